// Recurrent token mixers: the state of a request is carried in float from token to token, in a state slot.
//
// Both kernels walk the tokens of one request in order, whatever the step holds of it (a whole prompt, a portion, one
// decoded token), starting from the slot's state and leaving the new state there.  The chain of float operations of a
// channel therefore depends on the request's tokens only: not on how they were cut into steps nor on the batch.
// Projections come in the model's type T (bfloat16 when serving); gates, decays, the state and the norm are float.
#include "common.cuh"

namespace vob {

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
// The same for inputs of type T: behind 16-bit inputs the hardware's exponential and division (a few float units, far below
// the input's own rounding) take a quarter of the instructions.
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) { return sizeof(T) == 2 ? __fdividef(1.f, 1.f + __expf(-x)) : sigmoid_f(x); }
// f = l + (1 - l) sigmoid(pre + bias): one spelling for every kernel that needs the gate
__device__ __forceinline__ float forget_gate(float l, float pre, float bias) { return fmaf(1.f - l, sigmoid_f(pre + bias), l); }

// ---------------------------------------------------------------- minGRU
// zxg [tokens, 3W]: pre-activations of the gate z, of the candidate u and of the output gate g (no bias yet).
//   z = sigmoid(z + bz);  c = u + bx;  c = c >= 0 ? c + 1/2 : sigmoid(c);  s = (1 - z) s + z c;  out = s * silu(g)
// A block owns 32 channels of one request; neighbouring threads read neighbouring channels.  With NCH > 1 the request's
// tokens of this step are cut into NCH ranges, one per thread row: every row first folds its range into (A, B) with
// s_end = A s_start + B, the rows' starts follow from the state and the (A, B) before them, and a second walk writes
// the outputs.  A recurrence is a chain: without the cut a prompt of thousands of tokens runs on a thread per channel.
// The cut changes where a channel's additions are rounded, never what is computed.
struct GruStep { float z, c, g; };

template <typename T>
__device__ __forceinline__ GruStep gru_step(const T* row, int c, int W, float biasz, float biasx) {
  GruStep r;
  r.z = sigmoid_f(to_f<T>(row[c]) + biasz);
  const float u = to_f<T>(row[W + c]) + biasx;
  r.c = u >= 0.f ? u + 0.5f : sigmoid_f(u);
  r.g = to_f<T>(row[2 * W + c]);
  return r;
}

template <typename T, int NCH>
__global__ void __launch_bounds__(32 * NCH)
mingru_scan_kernel(const T* zxg, const T* __restrict__ bz, const T* __restrict__ bx, float* state,
                   const int* __restrict__ cu_q, const int* __restrict__ state_slots, T* out, int W,
                   int num_slots, int* err) {
  __shared__ float As[NCH][32], Bs[NCH][32];
  pdl_launch_dependents();
  const int b = blockIdx.y, lane = threadIdx.x, ch = threadIdx.y;
  const int c = min(blockIdx.x * 32 + lane, W - 1);
  const bool live = blockIdx.x * 32 + lane < W;
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  const int slot = state_slots[b];
  const float biasz = to_f<T>(bz[c]), biasx = to_f<T>(bx[c]);
  pdl_wait();
  if (t1 <= t0) return;
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0 && ch == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  const int per = (t1 - t0 + NCH - 1) / NCH;
  const int lo = min(t1, t0 + ch * per), hi = min(t1, lo + per);
  float s = state[(size_t)slot * W + c];
  if (NCH > 1) {
    float A = 1.f, B = 0.f;
#pragma unroll 4
    for (int t = lo; t < hi; ++t) {
      const GruStep g = gru_step<T>(zxg + (size_t)t * 3 * W, c, W, biasz, biasx);
      A *= 1.f - g.z;
      B = fmaf(g.z, g.c, (1.f - g.z) * B);
    }
    As[ch][lane] = A;
    Bs[ch][lane] = B;
    __syncthreads();
    for (int k = 0; k < ch; ++k) s = fmaf(As[k][lane], s, Bs[k][lane]);
  }
  // four tokens at a time: their loads are issued before the first store (the compiler cannot know that `out` is
  // another buffer, and would otherwise wait for every store before the next token's loads)
  int t = lo;
  for (; t + 4 <= hi; t += 4) {
    GruStep g[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) g[k] = gru_step<T>(zxg + (size_t)(t + k) * 3 * W, c, W, biasz, biasx);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      s = fmaf(g[k].z, g[k].c, (1.f - g[k].z) * s);
      if (live) out[(size_t)(t + k) * W + c] = from_f<T>(s * (g[k].g * sigmoid_f(g[k].g)));
    }
  }
  for (; t < hi; ++t) {
    const GruStep g = gru_step<T>(zxg + (size_t)t * 3 * W, c, W, biasz, biasx);
    s = fmaf(g.z, g.c, (1.f - g.z) * s);
    if (live) out[(size_t)t * W + c] = from_f<T>(s * (g.g * sigmoid_f(g.g)));
  }
  if (ch == NCH - 1 && live) state[(size_t)slot * W + c] = s;
}

// ---------------------------------------------------------------- a gated linear recurrence a channel (RG-LRU)
// u [tokens, W] of T (the convolution's output), gates float [tokens, blocks, 2, W / blocks] (pre-activations of r and i,
// block by block), y rows of y_stride elements (the other branch's projection):
//   r = sigmoid(r + br), i = sigmoid(i + bi), log a = -8 r softplus(lam), S = a S + sqrt(1 - a^2) i u,
//   out = S * gelu(y + by)                                 (the tanh form of gelu)
// 1 - a^2 = -expm1(2 log a): the difference would lose what a slow channel (a near 1) writes.  Cut along the tokens as minGRU.
struct LruStep { float a, b; };

template <typename T>
__device__ __forceinline__ LruStep lru_step(float gr, float gi, float u, float rate) {
  const float log_a = rate * sigmoid_t<T>(gr);
  return {expf(log_a), sqrtf(-expm1f(2.f * log_a)) * sigmoid_t<T>(gi) * u};
}

// A block owns LANES channels: 32, or 16 with twice the ranges where a long portion would otherwise leave SMs without a block.
template <typename T, int LANES, int NCH>
__global__ void __launch_bounds__(LANES * NCH)
lru_scan_kernel(const T* u, const float* gates, const T* y, long y_stride, const float* __restrict__ br, const float* __restrict__ bi,
                const float* __restrict__ lam, const float* __restrict__ by, float* state, long state_stride,
                const int* __restrict__ cu_q, const int* __restrict__ state_slots, T* out, int W, int per_block, int num_slots,
                int* err) {
  __shared__ float As[NCH][LANES], Bs[NCH][LANES];
  pdl_launch_dependents();
  const int b = blockIdx.y, lane = threadIdx.x, ch = threadIdx.y;
  const int c = min(blockIdx.x * LANES + lane, W - 1);
  const bool live = blockIdx.x * LANES + lane < W;
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  const int slot = state_slots[b];
  const float l = lam[c], biasr = br[c], biasi = bi[c], biasy = by[c];
  const float rate = -8.f * (fmaxf(l, 0.f) + log1pf(expf(-fabsf(l))));
  const size_t goff = (size_t)(c / per_block) * 2 * per_block + c % per_block;
  pdl_wait();
  if (t1 <= t0) return;
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0 && ch == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  const int per = (t1 - t0 + NCH - 1) / NCH;
  const int lo = min(t1, t0 + ch * per), hi = min(t1, lo + per);
  float s = state[(size_t)slot * state_stride + c];
  auto step = [&](int t) {
    const float* g = gates + (size_t)t * 2 * W + goff;
    return lru_step<T>(g[0] + biasr, g[per_block] + biasi, to_f<T>(u[(size_t)t * W + c]), rate);
  };
  if (NCH > 1) {
    float A = 1.f, B = 0.f;
#pragma unroll 4
    for (int t = lo; t < hi; ++t) {
      const LruStep g = step(t);
      A *= g.a;
      B = fmaf(g.a, B, g.b);
    }
    As[ch][lane] = A;
    Bs[ch][lane] = B;
    __syncthreads();
    for (int k = 0; k < ch; ++k) s = fmaf(As[k][lane], s, Bs[k][lane]);
    __syncthreads();
  }
  // four tokens at a time: their loads are issued before the first store
  for (int t = lo; t < hi; t += 4) {
    LruStep g[4];
    float yv[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int tk = min(t + k, hi - 1);
      g[k] = step(tk);
      yv[k] = to_f<T>(y[(size_t)tk * y_stride + c]) + biasy;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (t + k < hi) {
        s = fmaf(g[k].a, s, g[k].b);
        if (live) out[(size_t)(t + k) * W + c] = from_f<T>(s * gelu_tanh_f(yv[k]));
      }
  }
  if (ch == NCH - 1 && live) state[(size_t)slot * state_stride + c] = s;
}

// ---------------------------------------------------------------- matrix states with a gate a row
// One recurrence, three ways to make its numbers.  Per head, with a state M [dk, dv]:
//     M = diag(f) M + w v^T,   o = M^T q            f: what a row keeps, w: what is written into it, q: the read-out
// A SOURCE makes q, f, w and v of a token from its projected row:
//   HgrnSource       qfv [tokens, heads*dk | heads*dk | heads*dv]: q = silu(q), f = l + (1 - l) sigmoid(f + bf), w = 1 - f
//   GlaSource        q * scale, w = k, f = sigmoid(z + bz)^(1 / tau) = exp(-softplus(-(z + bz)) / tau), a number a head and row
//   LightningSource  q = silu(q), w = silu(k), v = silu(v), f = a fixed number a head
//   MlstmSource      q * scale, w = put * k, f = keep: two numbers a head and token (exponential gates, mlstm_gates below)
// A source with a NORMALISER carries one more column beside the head's dv, whose value is 1 at every token: n = diag(f) n + w.
// Its read-out n . q divides the head's outputs.  The column lies behind all heads' matrices, [heads, dk].
// Decoding, one token a request (matrix_scan_step): one block a (request, head) streams the state through registers once, 16 bytes
// an access; its first loads are in flight before the kernels ahead have finished (only an earlier step can have written the
// state, and a step begins with a copy of its index arrays, which lets nothing of the step before run on).  Short portions
// (matrix_scan_fused): one block a (request, head) holds the state in registers over the tokens: column j of a head's state M (dk
// floats) is shared by PARTS neighbouring lanes, R rows each.  Both take the head's norm and what the source puts behind it; the
// first may leave the bare o instead.  The fused walk's gates of HG_TT tokens are made by the whole block at once and parked in shared memory (rows padded so that the PARTS lanes of a column
// read different banks).
//
// Portions (matrix_scan_tile): a walker thread holds a tile of 8 rows x 8 columns of M in registers, as pairs of rows, so that
// every gate it reads from shared memory serves 8 columns and every multiply-add instruction two elements; ceil(dk / 8) lanes
// (a power of two) share 8 columns and halve their partial sums of o with every exchange.  Up to eight walker warps hold a
// head; eight loader warps make the gates of the next HG_TT tokens meanwhile, in the other of two buffers (named barriers:
// "full" when a buffer is ready, "empty" when its tokens have been walked).  o leaves in float and a norm kernel follows.
//
// A long portion is also cut along the tokens (`chunks` > 1, four launches): MODE 1 walks every range from a zero state
// and leaves its end state L; matrix_scan_range_decay takes the product F of every range's decays (a source with a normaliser has
// it made in MODE 1, by the warp that walks the normaliser); matrix_scan_join goes through the ranges in order,
// M_start(c+1) = diag(F_c) M_start(c) + L_c, leaves every range's start where its L was and the last state in the
// slot; MODE 2 walks the ranges again from their starts and writes the outputs.  Nearly twice the arithmetic, on as many more
// blocks as there are ranges.  MODE 0 is the walk from the slot's state to the slot's state in one launch.
constexpr int HG_TT = 16;

// index of gate i in a row of shared memory: four floats of padding after every 32, so that the lanes that share a column
// (32 or 64 rows apart) read different banks with 16-byte loads
__device__ __forceinline__ int hg_pad(int i) { return i + 4 * (i >> 5); }

struct ScanGates { float q, f, w; };

// What a head keeps by: a number a row and token, one number for all of a head's tokens, or a number a token for all its rows.
enum { DECAY_ROW = 0, DECAY_FIXED = 1, DECAY_TOKEN = 2 };

// What a source keeps of a (head, row) over the tokens, what it reads of a token, and what it makes of both.
template <typename T>
struct HgrnSource {
  static constexpr int DECAY = DECAY_ROW;
  static constexpr bool NORMALISER = false, HEAD_GATES = false;
  const T* rows;
  long width;
  const T* bf;
  const float* lower;
  int heads, dk, dv;
  struct Fixed { float l, bias; };
  struct Raw { float q, f; };
  __device__ __forceinline__ Fixed fixed(int h, int i) const { return {lower[h * dk + i], to_f<T>(bf[h * dk + i])}; }
  __device__ __forceinline__ Raw load(size_t t, int h, int i) const {
    const T* row = rows + t * width;
    return {to_f<T>(row[h * dk + i]), to_f<T>(row[(heads + h) * dk + i])};
  }
  __device__ __forceinline__ ScanGates make(const Raw& r, const Fixed& x) const {
    const float f = forget_gate(x.l, r.f, x.bias);
    return {r.q * sigmoid_t<T>(r.q), f, 1.f - f};
  }
  __device__ __forceinline__ float value(size_t t, int h, int c) const { return to_f<T>(rows[t * width + (size_t)2 * heads * dk + h * dv + c]); }
  __device__ __forceinline__ float decay(size_t t, int h, int i, const Fixed& x) const {
    return forget_gate(x.l, to_f<T>(rows[t * width + (size_t)(heads + h) * dk + i]), x.bias);
  }
  __device__ __forceinline__ float fixed_decay(int) const { return 0.f; }
  __device__ __forceinline__ float finish(float o, size_t, int, int) const { return o; }
};

// rows: q | k | v (heads*dk, heads*dk, heads*dv), the decay's pre-activations at z_off, the output gate at gate_off.
template <typename T>
struct GlaSource {
  static constexpr int DECAY = DECAY_ROW;
  static constexpr bool NORMALISER = false, HEAD_GATES = false;
  const T* rows;
  long width;
  const float* bias;       // [heads * dk]
  int heads, dk, dv, z_off, gate_off;
  float scale, inv_tau;
  struct Fixed { float bias; };
  struct Raw { float q, k, z; };
  __device__ __forceinline__ Fixed fixed(int h, int i) const { return {bias[h * dk + i]}; }
  __device__ __forceinline__ Raw load(size_t t, int h, int i) const {
    const T* row = rows + t * width;
    return {to_f<T>(row[h * dk + i]), to_f<T>(row[(heads + h) * dk + i]), to_f<T>(row[z_off + h * dk + i])};
  }
  // sigmoid(z)^(1/tau) by its logarithm: log sigmoid(z) = -softplus(-z) = min(z, 0) - log(1 + e^-|z|)
  __device__ __forceinline__ float keep(float z) const {
    if (sizeof(T) == 2) return __expf((fminf(z, 0.f) - __logf(1.f + __expf(-fabsf(z)))) * inv_tau);
    return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau);
  }
  __device__ __forceinline__ ScanGates make(const Raw& r, const Fixed& x) const { return {r.q * scale, keep(r.z + x.bias), r.k}; }
  __device__ __forceinline__ float value(size_t t, int h, int c) const { return to_f<T>(rows[t * width + (size_t)2 * heads * dk + h * dv + c]); }
  __device__ __forceinline__ float decay(size_t t, int h, int i, const Fixed& x) const {
    return keep(to_f<T>(rows[t * width + z_off + (size_t)h * dk + i]) + x.bias);
  }
  // behind the head's norm: times silu(gate)
  __device__ __forceinline__ float fixed_decay(int) const { return 0.f; }
  __device__ __forceinline__ float finish(float o, size_t t, int h, int c) const {
    const float g = to_f<T>(rows[t * width + gate_off + (size_t)h * dv + c]);
    return o * (g * sigmoid_f(g));
  }
};

// rows: q | k | v (heads*dk, heads*dk, heads*dv).
template <typename T>
struct LightningSource {
  static constexpr int DECAY = DECAY_FIXED;
  static constexpr bool NORMALISER = false, HEAD_GATES = false;
  const T* rows;
  long width;
  const float* decays;     // [heads]
  int heads, dk, dv;
  struct Fixed { float f; };
  struct Raw { float q, k; };
  __device__ __forceinline__ Fixed fixed(int h, int) const { return {decays[h]}; }
  __device__ __forceinline__ float fixed_decay(int h) const { return decays[h]; }
  __device__ __forceinline__ Raw load(size_t t, int h, int i) const {
    const T* row = rows + t * width;
    return {to_f<T>(row[h * dk + i]), to_f<T>(row[(heads + h) * dk + i])};
  }
  __device__ __forceinline__ ScanGates make(const Raw& r, const Fixed& x) const { return {r.q * sigmoid_t<T>(r.q), x.f, r.k * sigmoid_t<T>(r.k)}; }
  __device__ __forceinline__ float value(size_t t, int h, int c) const {
    const float v = to_f<T>(rows[t * width + (size_t)2 * heads * dk + h * dv + c]);
    return v * sigmoid_t<T>(v);
  }
  __device__ __forceinline__ float decay(size_t, int, int, const Fixed& x) const { return x.f; }
  __device__ __forceinline__ float finish(float o, size_t, int, int) const { return o; }
};

// ---- exponential gates
// Per head the pre-activations zi, zf (with biases) become log gates i = cap tanh(zi / cap), f = log sigmoid(cap tanh(zf / cap));
// with the running maximum m_t = max(f + m_{t-1}, i) a token keeps by exp(f + m_{t-1} - m_t) and writes by exp(i - m_t).  `floor`
// is exp(-m_t), the least that the normaliser's read-out counts as.
struct LogGates { float i, f; };
__device__ __forceinline__ LogGates log_gates(float zi, float zf, float cap) {
  const float x = cap * tanhf(zf / cap);
  return {cap * tanhf(zi / cap), fminf(x, 0.f) - log1pf(expf(-fabsf(x)))};
}
constexpr float MLSTM_EPS = 1e-6f;      // added to the normaliser

// rows: q | k | v (heads*dk, heads*dk, heads*dv), the pre-activations of i and f (heads each) at i_off and f_off, the output gate
// (heads*dv) at gate_off.  gates: float4 [tokens, heads] of (keep, put, floor, -), made by mlstm_gates_kernel for portions
// (GLOBAL), in the kernel itself for decoding.  A request's running maximum lies behind the normalisers, [heads].
template <typename T, bool GLOBAL>
struct MlstmSource {
  static constexpr int DECAY = DECAY_TOKEN;
  static constexpr bool NORMALISER = true, HEAD_GATES = !GLOBAL;
  const T* rows;
  long width;
  const float* bi;         // [heads]
  const float* bf;         // [heads]
  const float4* gates;
  float* nq;               // [tokens, heads] the normaliser's read-out
  int heads, dk, dv, i_off, f_off, gate_off;
  float scale, cap;
  struct Fixed {};
  struct Raw { float q, k; float2 g; };
  __device__ __forceinline__ Fixed fixed(int, int) const { return {}; }
  __device__ __forceinline__ float fixed_decay(int) const { return 0.f; }
  __device__ __forceinline__ Raw load(size_t t, int h, int i) const {
    const T* row = rows + t * width;
    return {to_f<T>(row[h * dk + i]), to_f<T>(row[(heads + h) * dk + i]),
            GLOBAL ? *reinterpret_cast<const float2*>(gates + t * heads + h) : make_float2(1.f, 1.f)};
  }
  __device__ __forceinline__ ScanGates make(const Raw& r, const Fixed&) const { return {r.q * scale, r.g.x, r.k * r.g.y}; }
  __device__ __forceinline__ float token_decay(size_t t, int h) const { return gates[t * heads + h].x; }
  __device__ __forceinline__ float value(size_t t, int h, int c) const { return to_f<T>(rows[t * width + (size_t)2 * heads * dk + h * dv + c]); }
  __device__ __forceinline__ LogGates pre(size_t t, int h) const {
    const T* row = rows + t * width;
    return log_gates(to_f<T>(row[i_off + h]) + bi[h], to_f<T>(row[f_off + h]) + bf[h], cap);
  }
  // behind the head's norm: times sigmoid(gate)
  __device__ __forceinline__ float finish(float o, size_t t, int h, int c) const {
    return o * sigmoid_f(to_f<T>(rows[t * width + gate_off + (size_t)h * dv + c]));
  }
};

// The gates of a step's portions, one block a (request, head).  m over a range of tokens is max(a + m, b) with a the sum of its f:
// every thread folds its own range, the block scans the folds, and every thread walks its range again from its start.  A
// range's last maximum is the next range's start by construction, so what a token keeps and writes refers to one and the same m.
constexpr int MG_NT = 1024;
constexpr int MG_HELD = 4;      // tokens of a thread whose log gates stay in registers between the two walks

template <typename T>
__global__ void __launch_bounds__(MG_NT)
mlstm_gates_kernel(const MlstmSource<T, true> src, float4* gates, float* state, long state_stride, const int* __restrict__ cu_q,
                   const int* __restrict__ state_slots, int num_slots, int* err) {
  __shared__ float wa[MG_NT / 32], wb[MG_NT / 32], starts[MG_NT + 1];
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = cu_q[b], t1 = cu_q[b + 1], slot = state_slots[b];
  pdl_wait();
  if (t1 <= t0) return;
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  float* kept = state + (size_t)slot * state_stride + (size_t)src.heads * src.dk * (src.dv + 1) + h;
  const float first = *kept;
  const int per = (t1 - t0 + MG_NT - 1) / MG_NT;
  const int lo = min(t1, t0 + (int)threadIdx.x * per), hi = min(t1, lo + per);
  float a = 0.f, m = -INFINITY;
  LogGates held[MG_HELD];
#pragma unroll
  for (int k = 0; k < MG_HELD; ++k)
    if (lo + k < hi) held[k] = src.pre((size_t)(lo + k), h);
#pragma unroll
  for (int k = 0; k < MG_HELD; ++k)
    if (lo + k < hi) {
      a += held[k].f;
      m = fmaxf(held[k].f + m, held[k].i);
    }
#pragma unroll 2
  for (int t = lo + MG_HELD; t < hi; ++t) {
    const LogGates g = src.pre((size_t)t, h);
    a += g.f;
    m = fmaxf(g.f + m, g.i);
  }
  // inclusive scan over the threads: what a fold (a, m) makes of a fold (a', m') before it
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const float pa = __shfl_up_sync(0xffffffffu, a, d), pm = __shfl_up_sync(0xffffffffu, m, d);
    if (lane >= d) {
      m = fmaxf(a + pm, m);
      a += pa;
    }
  }
  if (lane == 31) { wa[warp] = a; wb[warp] = m; }
  __syncthreads();
  float start = first;
  for (int w = 0; w < warp; ++w) start = fmaxf(wa[w] + start, wb[w]);
  starts[threadIdx.x + 1] = fmaxf(a + start, m);
  if (threadIdx.x == 0) starts[0] = first;
  __syncthreads();
  m = starts[threadIdx.x];
  const float last = starts[threadIdx.x + 1];
  auto put = [&](int t, const LogGates& g) {
    const float next = t + 1 < hi ? fmaxf(g.f + m, g.i) : last;
    gates[(size_t)t * src.heads + h] = make_float4(expf(g.f + m - next), expf(g.i - next), expf(-next), 0.f);
    m = next;
  };
#pragma unroll
  for (int k = 0; k < MG_HELD; ++k)
    if (lo + k < hi) put(lo + k, held[k]);
#pragma unroll 2
  for (int t = lo + MG_HELD; t < hi; ++t) put(t, src.pre((size_t)t, h));
  if (hi == t1 && lo < hi) *kept = m;
}

// ---- decoding: a block a (request, head)
template <typename T, typename SOURCE, int R, int PARTS>
__global__ void __launch_bounds__(R > 32 ? 256 : 512)
matrix_scan_fused_kernel(const SOURCE src, const float* __restrict__ nw, float* state, long state_stride, const int* __restrict__ cu_q,
                         const int* __restrict__ state_slots, T* out, int heads, int dk, int dv, float eps, int num_slots, int* err) {
  extern __shared__ float4 sm4[];
  float* sm = reinterpret_cast<float*>(sm4);
  const int gate_row = hg_pad(R * PARTS);
  const int cols = blockDim.x / PARTS;
  float* qs = sm;                        // [HG_TT][gate_row]
  float* fs = qs + HG_TT * gate_row;     // [HG_TT][gate_row]  f
  float* gs = fs + HG_TT * gate_row;     // [HG_TT][gate_row]  w
  float* vs = gs + HG_TT * gate_row;     // [HG_TT][cols]
  float* os = vs + HG_TT * cols;         // [HG_TT][cols]
  __shared__ float keeps[SOURCE::HEAD_GATES ? HG_TT : 1], puts[SOURCE::HEAD_GATES ? HG_TT : 1], floors[SOURCE::HEAD_GATES ? HG_TT : 1];
  __shared__ float norms[SOURCE::HEAD_GATES ? R * PARTS : 1];      // the head's normaliser: warp 0 walks it, a lane its own rows
  pdl_launch_dependents();
  const int part = threadIdx.x % PARTS, j = threadIdx.x / PARTS;
  const int h = blockIdx.x, b = blockIdx.y;
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  const int slot = state_slots[b];
  pdl_wait();
  if (t1 <= t0) return;
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  const int i0 = part * R;
  float* mine = state + (size_t)slot * state_stride + ((size_t)h * dk + i0) * dv + j;
  float M[R];
#pragma unroll
  for (int i = 0; i < R; ++i) M[i] = (i0 + i < dk && j < dv) ? mine[(size_t)i * dv] : 0.f;
  float* norm = nullptr;                   // in the slot: the head's normaliser, the running maximum of its gates
  float* kept = nullptr;
  float run = 0.f;
  if constexpr (SOURCE::HEAD_GATES) {
    norm = state + (size_t)slot * state_stride + (size_t)heads * dk * dv + (size_t)h * dk;
    kept = state + (size_t)slot * state_stride + (size_t)heads * dk * (dv + 1) + h;
    run = *kept;
    if (threadIdx.x < 32)
      for (int i = threadIdx.x; i < dk; i += 32) norms[i] = norm[i];
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  // the gates of a tile: thread rows over tokens, thread columns over gates (one division, here)
  const int gate_lanes = min(dk, (int)blockDim.x), gate_step = blockDim.x / gate_lanes;
  const int gate_i = threadIdx.x % gate_lanes, gate_t = threadIdx.x / gate_lanes < gate_step ? threadIdx.x / gate_lanes : HG_TT;
  for (int ts = t0; ts < t1; ts += HG_TT) {
    const int n = min(HG_TT, t1 - ts);
    if constexpr (SOURCE::HEAD_GATES) {
      // warp 0: a lane makes a token's log gates, the maxima go from lane to lane, a lane makes its token's factors
      if (warp == 0) {
        const LogGates lg = src.pre((size_t)(ts + min(lane, n - 1)), h);
        float before = run, now = run;
        for (int tt = 0; tt < n; ++tt) {
          const float next = fmaxf(__shfl_sync(0xffffffffu, lg.f, tt) + run, __shfl_sync(0xffffffffu, lg.i, tt));
          if (lane == tt) { before = run; now = next; }
          run = next;
        }
        if (lane < n) {
          keeps[lane] = expf(lg.f + before - now);
          puts[lane] = expf(lg.i - now);
          floors[lane] = expf(-now);
        }
      }
      __syncthreads();
    }
    for (int i = gate_i; i < dk; i += gate_lanes) {
      const typename SOURCE::Fixed fx = src.fixed(h, i);
      for (int tt = gate_t; tt < n; tt += gate_step) {
        ScanGates g = src.make(src.load((size_t)(ts + tt), h, i), fx);
        if constexpr (SOURCE::HEAD_GATES) {
          g.f = keeps[tt];
          g.w *= puts[tt];
        }
        qs[tt * gate_row + hg_pad(i)] = g.q;
        fs[tt * gate_row + hg_pad(i)] = g.f;
        gs[tt * gate_row + hg_pad(i)] = g.w;
      }
    }
    for (int idx = threadIdx.x; idx < n * cols; idx += blockDim.x) {
      const int tt = idx / cols, c = idx % cols;
      vs[idx] = c < dv ? src.value((size_t)(ts + tt), h, c) : 0.f;
    }
    __syncthreads();
    if constexpr (SOURCE::HEAD_GATES) {
      // what a token's outputs are divided by takes its floor's place
      if (warp == 0)
        for (int tt = 0; tt < n; ++tt) {
          float s = 0.f;
          for (int i = lane; i < dk; i += 32) {
            const int at = tt * gate_row + hg_pad(i);
            const float x = fmaf(fs[at], norms[i], gs[at]);
            norms[i] = x;
            s = fmaf(x, qs[at], s);
          }
          s = warp_sum(s);
          if (lane == 0) floors[tt] = fmaxf(fabsf(s), floors[tt]) + MLSTM_EPS;
          __syncwarp();
        }
    }
#pragma unroll 2
    for (int tt = 0; tt < n; ++tt) {
      float o = 0.f;
      const float v = vs[tt * cols + j];
      const float* fr = fs + tt * gate_row + hg_pad(i0);
      const float* gr = gs + tt * gate_row + hg_pad(i0);
      const float* qr = qs + tt * gate_row + hg_pad(i0);
#pragma unroll
      for (int i = 0; i < R; i += 4) {
        const float4 f4 = *reinterpret_cast<const float4*>(fr + hg_pad(i));      // hg_pad(i0 + i) = hg_pad(i0) + hg_pad(i)
        const float4 g4 = *reinterpret_cast<const float4*>(gr + hg_pad(i));
        const float4 q4 = *reinterpret_cast<const float4*>(qr + hg_pad(i));
        const float fv[4] = {f4.x, f4.y, f4.z, f4.w}, gv[4] = {g4.x, g4.y, g4.z, g4.w}, qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (i0 + i + k < dk) {
            M[i + k] = fmaf(fv[k], M[i + k], gv[k] * v);
            o = fmaf(M[i + k], qv[k], o);
          }
      }
#pragma unroll
      for (int d = 1; d < PARTS; d <<= 1) o += __shfl_xor_sync(0xffffffffu, o, d);
      if (part == 0) os[tt * cols + j] = o;
    }
    __syncthreads();
    for (int tt = warp; tt < n; tt += nwarps) {
      float ss = 0.f, unit = 1.f;
      if constexpr (SOURCE::HEAD_GATES) unit = 1.f / floors[tt];
      for (int c = lane; c < dv; c += 32) {
        const float o = os[tt * cols + c] * unit;
        ss += o * o;
      }
      const float denom = sqrtf(warp_sum(ss) / (float)dv + eps);
      const float* gain = SOURCE::HEAD_GATES ? nw + (size_t)h * dv : nw;      // a gain for all heads' elements, or one head's
      for (int c = lane; c < dv; c += 32)
        out[(size_t)(ts + tt) * heads * dv + h * dv + c] =
            from_f<T>(src.finish(os[tt * cols + c] * unit / denom * gain[c], (size_t)(ts + tt), h, c));
    }
    __syncthreads();
  }
  if (j < dv) {
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (i0 + i < dk) mine[(size_t)i * dv] = M[i];
  }
  if constexpr (SOURCE::HEAD_GATES) {
    if (threadIdx.x < 32)
      for (int i = threadIdx.x; i < dk; i += 32) norm[i] = norms[i];
    if (threadIdx.x == 0) *kept = run;
  }
}


// ---- decoding: the state passes through registers once a token
// A thread has VEC neighbouring columns and every `groups`-th row, U rows in flight; the groups' shares of o meet in shared memory.
template <typename T, typename SOURCE, int VEC, int NT>
__global__ void __launch_bounds__(NT, 1024 / NT)
matrix_scan_step_kernel(const SOURCE src, const float* __restrict__ nw, float* state, long state_stride, const int* __restrict__ cu_q,
                        const int* __restrict__ state_slots, T* out, float* raw, int heads, int dk, int dv, float eps, int num_slots,
                        int* err) {
  constexpr int U = 8;
  extern __shared__ float4 sm4[];
  __shared__ float red[NT / 32];
  float* qs = reinterpret_cast<float*>(sm4);      // [dk] each
  float* fs = qs + dk;
  float* ws = fs + dk;
  float* os = ws + dk;                            // [groups][dv]
  pdl_launch_dependents();
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const int t0 = cu_q[b], t1 = cu_q[b + 1], slot = state_slots[b];
  const bool ok = t1 > t0 && slot >= 0 && slot < num_slots;
  const int C = dv / VEC, groups = NT / C;
  const int c = tid % C * VEC, g = tid / C;
  const bool have = g < groups;
  float* whole = ok ? state + (size_t)slot * state_stride : nullptr;
  float* mine = ok ? whole + (size_t)h * dk * dv + c : nullptr;
  float m[U][VEC];
  auto load_rows = [&](int r0) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int r = r0 + u * groups + g;
      if (have && r < dk) {
        if constexpr (VEC == 4) load4(mine + (size_t)r * dv, m[u]);
        else m[u][0] = mine[(size_t)r * dv];
      }
    }
  };
  float n_row = 0.f, run = 0.f;                   // the normaliser's row tid, the running maximum
  float* norm = nullptr;
  float* kept = nullptr;
  const typename SOURCE::Fixed fx = src.fixed(h, min(tid, dk - 1));
  if (ok) {
    load_rows(0);
    if constexpr (SOURCE::NORMALISER) {
      norm = whole + (size_t)heads * dk * dv + (size_t)h * dk + tid;
      kept = whole + (size_t)heads * dk * (dv + 1) + h;
      if (tid < dk) n_row = *norm;
      run = *kept;
    }
  }
  pdl_wait();
  if (!ok) {
    if (t1 > t0 && tid == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  for (int t = t0; t < t1; ++t) {
    float floor = 0.f, share = 0.f;
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = src.value((size_t)t, h, c + e);
    ScanGates gate = {0.f, 0.f, 0.f};
    if (tid < dk) gate = src.make(src.load((size_t)t, h, tid), fx);
    if constexpr (SOURCE::HEAD_GATES) {
      const LogGates lg = src.pre((size_t)t, h);
      const float next = fmaxf(lg.f + run, lg.i);
      gate.f = expf(lg.f + run - next);
      gate.w *= expf(lg.i - next);
      floor = expf(-next);
      run = next;
    }
    if (tid < dk) {
      qs[tid] = gate.q;
      fs[tid] = gate.f;
      ws[tid] = gate.w;
      if constexpr (SOURCE::NORMALISER) {
        n_row = fmaf(gate.f, n_row, gate.w);
        share = n_row * gate.q;
      }
    }
    __syncthreads();
    float o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = 0.f;
    for (int r0 = 0; r0 < dk; r0 += U * groups) {
      if (r0 > 0 || t > t0) load_rows(r0);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * groups + g;
        if (have && r < dk) {
          const float f = fs[r], w = ws[r], q = qs[r];
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            m[u][e] = fmaf(f, m[u][e], w * v[e]);
            o[e] = fmaf(m[u][e], q, o[e]);
          }
          if constexpr (VEC == 4) store4(mine + (size_t)r * dv, m[u]);
          else mine[(size_t)r * dv] = m[u][0];
        }
      }
    }
    if (have) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) os[g * dv + c + e] = o[e];
    }
    float unit = 1.f;
    if constexpr (SOURCE::NORMALISER) unit = 1.f / (fmaxf(fabsf(block_sum<NT>(share, red)), floor) + MLSTM_EPS);
    else __syncthreads();
    float ss = 0.f;
    for (int j = tid; j < dv; j += NT) {
      float s = os[j];
      for (int k = 1; k < groups; ++k) s += os[k * dv + j];
      s *= unit;
      os[j] = s;
      ss = fmaf(s, s, ss);
    }
    const size_t row = (size_t)t * heads * dv + (size_t)h * dv;
    if (raw) {
      for (int j = tid; j < dv; j += NT) raw[row + j] = os[j];
    } else {
      const float denom = sqrtf(block_sum<NT>(ss, red) / (float)dv + eps);
      const float* gain = SOURCE::HEAD_GATES ? nw + (size_t)h * dv : nw;
      for (int j = tid; j < dv; j += NT) out[row + j] = from_f<T>(src.finish(os[j] / denom * gain[j], (size_t)t, h, j));
    }
    if (t + 1 < t1) __syncthreads();
  }
  if constexpr (SOURCE::NORMALISER) {
    if (tid < dk) *norm = n_row;
    if (tid == 0) *kept = run;
  }
}

// ---- portions: walkers and loaders
constexpr int MS_LOADERS = 256, MS_MAX_WALKERS = 256;
constexpr int MS_R = 8, MS_C = 8;      // a walker's rows and columns

// Where row i of a head lies among the PARTS * 8 gates of a token in shared memory: the first four rows of every part, then the
// last four, so that the 16-byte reads of neighbouring parts are neighbours.
template <int PARTS>
__device__ __forceinline__ int tile_index(int i) { return (((i & 7) >> 2) * PARTS + (i >> 3)) * 4 + (i & 3); }

// OUT: outputs are made (MODE 0 and 2 above); `mode` says where the walk starts and what it leaves.
template <typename SOURCE, int PARTS, bool OUT>
__global__ void __launch_bounds__(MS_LOADERS + MS_MAX_WALKERS, 1)
matrix_scan_tile_kernel(const SOURCE src, float* state, long state_stride, const int* __restrict__ cu_q,
                        const int* __restrict__ state_slots, float* raw, float* ends, int heads, int dk, int dv, int col_blocks,
                        int num_slots, int mode, int* err) {
  constexpr int W = PARTS * MS_R;              // gates of a token, rows past dk are zeros
  constexpr bool ROWS = SOURCE::DECAY == DECAY_ROW;      // a gate f a row lies in shared memory
  constexpr int KINDS = ROWS ? 3 : 2;                    // rows of gates a token
  extern __shared__ float4 sm4[];
  const int walkers = blockDim.x - MS_LOADERS, threads = blockDim.x;
  const int cols = walkers / PARTS * MS_C;     // columns of this block
  const int buffer = HG_TT * (KINDS * W + cols + (SOURCE::DECAY == DECAY_TOKEN ? 1 : 0));
  float* sm = reinterpret_cast<float*>(sm4);
  pdl_launch_dependents();
  const int h = blockIdx.x / col_blocks, c0 = blockIdx.x % col_blocks * cols;
  const int b = blockIdx.y, chunk = blockIdx.z, chunks = gridDim.z;
  const int q0 = cu_q[b], q1 = cu_q[b + 1];
  const int slot = state_slots[b];
  pdl_wait();
  if (q1 <= q0) return;
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, VOB_ERR_SLOT);
    return;
  }
  const int per = (q1 - q0 + chunks - 1) / chunks;
  const int t0 = min(q1, q0 + chunk * per), t1 = min(q1, t0 + per);
  const int tiles = (t1 - t0 + HG_TT - 1) / HG_TT;
  // where the walk's matrices start and end: the slot, or the range's place
  float* whole = mode == 0 ? state + (size_t)slot * state_stride
                           : ends + ((size_t)b * chunks + chunk) * ((size_t)heads * dk * (dv + (SOURCE::NORMALISER ? 1 : 0)));
  if ((int)threadIdx.x >= walkers) {
    // ------------------------------------------------ loaders
    const int tid = threadIdx.x - walkers;
    const int gate_lanes = min(dk, MS_LOADERS), gate_step = MS_LOADERS / gate_lanes;
    const int gate_i = tid % gate_lanes, gate_t = tid / gate_lanes < gate_step ? tid / gate_lanes : HG_TT;
    // rows past dk: zeros in both buffers, once
    for (int k = 0; k < 2; ++k)
      for (int idx = tid; idx < HG_TT * (W - dk); idx += MS_LOADERS) {
        float* q = sm + k * buffer + idx / (W - dk) * W + tile_index<PARTS>(dk + idx % (W - dk));
        q[0] = 0.f;
        q[HG_TT * W] = 0.f;
        if (ROWS) q[2 * HG_TT * W] = 0.f;
      }
    // the head's normaliser: the first loader warp walks it, a tile when its gates are there; a lane holds eight rows as a walker
    // does (groups of PARTS lanes hold copies)
    const bool norm_warp = SOURCE::NORMALISER && c0 == 0 && tid < 32;
    float* norm = whole + (size_t)heads * dk * dv + (size_t)h * dk + tid % PARTS * MS_R;
    f32x2 n2[MS_R / 2];
    float kept = 1.f;            // the product of the range's decays (one number a head)
    if constexpr (SOURCE::NORMALISER) {
      const int live = OUT && norm_warp ? dk - tid % PARTS * MS_R : 0;
#pragma unroll
      for (int p = 0; p < MS_R / 2; ++p) n2[p] = pack2(2 * p < live ? norm[2 * p] : 0.f, 2 * p + 1 < live ? norm[2 * p + 1] : 0.f);
    }
    for (int k = 0; k < tiles; ++k) {
      float* qs = sm + (k & 1) * buffer;       // [HG_TT][W] q
      float* ws = qs + HG_TT * W;              // [HG_TT][W] w
      float* fs = ws + HG_TT * W;              // [HG_TT][W] f (not where a head's rows share it)
      float* vs = qs + HG_TT * KINDS * W;      // [HG_TT][cols], behind it [HG_TT] f where it is a number a token
      const int ts = t0 + k * HG_TT, n = min(HG_TT, t1 - ts);
      if (k >= 2) named_sync(3 + (k & 1), threads);      // the walkers have left this buffer
      for (int i = gate_i; i < dk; i += gate_lanes) {
        const typename SOURCE::Fixed fx = src.fixed(h, i);
        const int at = tile_index<PARTS>(i);
        // eight tokens' loads are issued before the first of them is used
        for (int tb = gate_t; tb < n; tb += 8 * gate_step) {
          typename SOURCE::Raw raws[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) raws[e] = src.load((size_t)(ts + min(tb + e * gate_step, n - 1)), h, i);
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int tt = tb + e * gate_step;
            if (tt < n) {
              const ScanGates g = src.make(raws[e], fx);
              if (OUT) qs[tt * W + at] = g.q;
              ws[tt * W + at] = g.w;
              if (ROWS) fs[tt * W + at] = g.f;
            }
          }
        }
      }
      if constexpr (SOURCE::DECAY == DECAY_TOKEN) {
        if (tid < n) vs[HG_TT * cols + tid] = src.token_decay((size_t)(ts + tid), h);
      }
      // (a thread keeps its column, eight tokens' loads in flight)
      const int v_lanes = min(cols, MS_LOADERS), v_step = MS_LOADERS / v_lanes;
      for (int c = tid % v_lanes; c < cols; c += v_lanes)
        for (int tb = tid / v_lanes; tb < n; tb += 8 * v_step) {
          float v[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) v[e] = c0 + c < dv ? src.value((size_t)(ts + min(tb + e * v_step, n - 1)), h, c0 + c) : 0.f;
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (tb + e * v_step < n) vs[(tb + e * v_step) * cols + c] = v[e];
        }
      __threadfence_block();
      // (the loaders meet, so that the first of their warps may read the tile; they cannot come back to this buffer before it has
      // met them at the next tile)
      if constexpr (SOURCE::NORMALISER) named_sync(5, MS_LOADERS);
      named_arrive(1 + (k & 1), threads);
      if constexpr (SOURCE::NORMALISER) {
        if (norm_warp) {
#pragma unroll 4
          for (int tt = 0; tt < n; ++tt) {
            const float f = vs[HG_TT * cols + tt];
            const f32x2 keep = pack2(f, f);
            f32x2 s2 = 0ull;
            kept *= f;
#pragma unroll
            for (int p = 0; p < 2; ++p) {
              const int at = tt * W + (p * PARTS + tid % PARTS) * 4;
              const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(ws + at);
              n2[2 * p] = fma2(keep, n2[2 * p], w.x);
              n2[2 * p + 1] = fma2(keep, n2[2 * p + 1], w.y);
              if (OUT) {
                const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(qs + at);
                s2 = fma2(n2[2 * p], q.x, s2);
                s2 = fma2(n2[2 * p + 1], q.y, s2);
              }
            }
            if (OUT) {
              const float2 s = unpack2(s2);
              float sum = s.x + s.y;
#pragma unroll
              for (int d = 1; d < PARTS; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
              if (tid == 0) src.nq[(size_t)(ts + tt) * heads + h] = sum;
            }
          }
        }
      }
    }
    if constexpr (SOURCE::NORMALISER) {
      if (norm_warp && tid < PARTS && mode != 2) {
        const int live = dk - tid * MS_R;
#pragma unroll
        for (int p = 0; p < MS_R / 2; ++p) {
          const float2 x = unpack2(n2[p]);
          if (2 * p < live) norm[2 * p] = x.x;
          if (2 * p + 1 < live) norm[2 * p + 1] = x.y;
        }
        // (where matrix_scan_range_decay would leave it)
        if (mode == 1) {
          float* F = ends + (size_t)gridDim.y * chunks * heads * dk * (dv + 1) + (((size_t)b * chunks + chunk) * heads + h) * dk;
          for (int i = tid; i < dk; i += PARTS) F[i] = kept;
        }
      }
    }
    return;
  }
  // -------------------------------------------------- walkers
  const int part = threadIdx.x % PARTS, group = threadIdx.x / PARTS;
  const int j0 = c0 + group * MS_C, i0 = part * MS_R;
  float* mine = whole + (size_t)h * dk * dv;
  // (a head's matrix starts on a 16-byte boundary where the state's rows do)
  const bool wide = dv % 4 == 0 && (((uintptr_t)mine) & 15) == 0;
  f32x2 M[MS_C][MS_R / 2];
#pragma unroll
  for (int r = 0; r < MS_R; r += 2) {
    float a[2][MS_C];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = i0 + r + e;
      const float* row = mine + (size_t)i * dv + j0;
#pragma unroll
      for (int c = 0; c < MS_C; c += 4) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (OUT && i < dk) {
          if (wide) {
            if (j0 + c < dv) x = *reinterpret_cast<const float4*>(row + c);
          } else {
            if (j0 + c < dv) x.x = row[c];
            if (j0 + c + 1 < dv) x.y = row[c + 1];
            if (j0 + c + 2 < dv) x.z = row[c + 2];
            if (j0 + c + 3 < dv) x.w = row[c + 3];
          }
        }
        a[e][c] = x.x; a[e][c + 1] = x.y; a[e][c + 2] = x.z; a[e][c + 3] = x.w;
      }
    }
#pragma unroll
    for (int c = 0; c < MS_C; ++c) M[c][r / 2] = pack2(a[0][c], a[1][c]);
  }
  f32x2 f2[ROWS ? MS_R / 2 : 1];
  if (SOURCE::DECAY == DECAY_FIXED) {
    const float f = src.fixed_decay(h);
    f2[0] = pack2(f, f);
  }
  // the columns whose sums end in this lane
  constexpr int HALVINGS = PARTS >= 8 ? 3 : (PARTS >= 4 ? 2 : (PARTS >= 2 ? 1 : 0));
  constexpr int OWN = MS_C >> HALVINGS;
  int own = 0;
#pragma unroll
  for (int k = 0; k < HALVINGS; ++k)
    if (part & (1 << k)) own += MS_C >> (k + 1);
  const bool writes = PARTS <= 8 || part < 8;
  for (int k = 0; k < tiles; ++k) {
    const float* qs = sm + (k & 1) * buffer;
    const float* ws = qs + HG_TT * W;
    const float* fs = ws + HG_TT * W;
    const float* vs = qs + HG_TT * KINDS * W;
    const int ts = t0 + k * HG_TT, n = min(HG_TT, t1 - ts);
    named_sync(1 + (k & 1), threads);
#pragma unroll 1
    for (int tt = 0; tt < n; ++tt) {
      f32x2 w2[MS_R / 2], q2[MS_R / 2];
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        const int at = tt * W + (p * PARTS + part) * 4;
        const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(ws + at);
        w2[2 * p] = w.x; w2[2 * p + 1] = w.y;
        if (OUT) {
          const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(qs + at);
          q2[2 * p] = q.x; q2[2 * p + 1] = q.y;
        }
        if (ROWS) {
          const ulonglong2 f = *reinterpret_cast<const ulonglong2*>(fs + at);
          f2[ROWS ? 2 * p : 0] = f.x; f2[ROWS ? 2 * p + 1 : 0] = f.y;
        }
      }
      if (SOURCE::DECAY == DECAY_TOKEN) {
        const float f = vs[HG_TT * cols + tt];
        f2[0] = pack2(f, f);
      }
      float v[MS_C], o[MS_C];
      {
        const float4* v4 = reinterpret_cast<const float4*>(vs + tt * cols + group * MS_C);
        const float4 a = v4[0], c = v4[1];
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = c.x; v[5] = c.y; v[6] = c.z; v[7] = c.w;
      }
#pragma unroll
      for (int c = 0; c < MS_C; ++c) {
        const f32x2 v2 = pack2(v[c], v[c]);
        f32x2 o2 = 0ull;
#pragma unroll
        for (int p = 0; p < MS_R / 2; ++p) {
          M[c][p] = fma2(f2[ROWS ? p : 0], M[c][p], mul2(w2[p], v2));
          if (OUT) o2 = p == 0 ? mul2(M[c][p], q2[p]) : fma2(M[c][p], q2[p], o2);
        }
        if (OUT) {
          const float2 s = unpack2(o2);
          o[c] = s.x + s.y;
        }
      }
      if (OUT) {
        // every exchange halves the columns a lane still sums, until each has its own
#pragma unroll
        for (int e = 0; e < HALVINGS; ++e) {
          const int half = MS_C >> (e + 1);
          const bool upper = part & (1 << e);
#pragma unroll
          for (int c = 0; c < MS_C / 2; ++c)
            if (c < half) {
              const float give = upper ? o[c] : o[c + half], keep = upper ? o[c + half] : o[c];
              o[c] = keep + __shfl_xor_sync(0xffffffffu, give, 1 << e);
            }
        }
#pragma unroll
        for (int d = 8; d < PARTS; d <<= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], d);
        if (writes) {
          float* dst = raw + (size_t)(ts + tt) * heads * dv + (size_t)h * dv + j0 + own;
#pragma unroll
          for (int c = 0; c < OWN; ++c)
            if (j0 + own + c < dv) dst[c] = o[c];
        }
      }
    }
    if (k + 2 < tiles) named_arrive(3 + (k & 1), threads);
  }
  if (mode == 2) return;
#pragma unroll
  for (int r = 0; r < MS_R; r += 2) {
    float a[2][MS_C];
#pragma unroll
    for (int c = 0; c < MS_C; ++c) {
      const float2 x = unpack2(M[c][r / 2]);
      a[0][c] = x.x;
      a[1][c] = x.y;
    }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = i0 + r + e;
      if (i >= dk) continue;
      float* row = mine + (size_t)i * dv + j0;
#pragma unroll
      for (int c = 0; c < MS_C; c += 4) {
        if (wide) {
          if (j0 + c < dv) *reinterpret_cast<float4*>(row + c) = make_float4(a[e][c], a[e][c + 1], a[e][c + 2], a[e][c + 3]);
        } else {
#pragma unroll
          for (int d = 0; d < 4; ++d)
            if (j0 + c + d < dv) row[c + d] = a[e][c + d];
        }
      }
    }
  }
}

// gates[b][c][h][i] = the product of the forget gates of range c of request b: what an end state of that range owes to its start.
// A block takes 32 gates of one range; its eight warps take every eighth token, and their partial products are multiplied
// in the order of the warps.
template <typename SOURCE>
__global__ void __launch_bounds__(256)
matrix_scan_range_decay_kernel(const SOURCE src, float* gates, const int* __restrict__ cu_q, int heads, int dk) {
  __shared__ float part[8][32];
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, chunk = blockIdx.z, chunks = gridDim.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int e = min(blockIdx.x * 32 + lane, heads * dk - 1);      // (head, i)
  const int q0 = cu_q[b], q1 = cu_q[b + 1];
  if (q1 <= q0) return;
  const int per = (q1 - q0 + chunks - 1) / chunks;
  const int t0 = min(q1, q0 + chunk * per), t1 = min(q1, t0 + per);
  const typename SOURCE::Fixed fx = src.fixed(e / dk, e % dk);
  float F = 1.f;
#pragma unroll 4
  for (int t = t0 + warp; t < t1; t += 8) F *= src.decay((size_t)t, e / dk, e % dk, fx);
  part[warp][lane] = F;
  __syncthreads();
  if (warp == 0 && blockIdx.x * 32 + lane < heads * dk) {
    F = part[0][lane];
#pragma unroll
    for (int k = 1; k < 8; ++k) F *= part[k][lane];
    gates[((size_t)b * chunks + chunk) * heads * dk + e] = F;
  }
}

// One thread per element of a request's state: through the ranges in order, start(c) takes the place of L_c.  All of a
// thread's loads are issued before its first store (at most HG_MAX_CHUNKS ranges), or every store would wait for a load.
constexpr int HG_MAX_CHUNKS = 16;

__global__ void matrix_scan_join_kernel(float* state, long state_stride, float* ends, const float* gates, const int* __restrict__ cu_q,
                                  const int* __restrict__ state_slots, int chunks, int heads, int dk, int dv, long per,
                                  int num_slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y;
  const long e = (long)blockIdx.x * blockDim.x + threadIdx.x, matrices = (long)heads * dk * dv;
  const int slot = state_slots[b];
  if (e >= per || cu_q[b + 1] <= cu_q[b] || slot < 0 || slot >= num_slots) return;
  const long row = e < matrices ? e / dv : e - matrices;      // (head, i); behind the matrices a column of normalisers
  float L[HG_MAX_CHUNKS], F[HG_MAX_CHUNKS];
#pragma unroll
  for (int c = 0; c < HG_MAX_CHUNKS; ++c)
    if (c < chunks) {
      L[c] = ends[((size_t)b * chunks + c) * per + e];
      F[c] = gates[((size_t)b * chunks + c) * heads * dk + row];
    }
  float M = state[(size_t)slot * state_stride + e];
#pragma unroll
  for (int c = 0; c < HG_MAX_CHUNKS; ++c)
    if (c < chunks) {
      ends[((size_t)b * chunks + c) * per + e] = M;
      M = fmaf(F[c], M, L[c]);
    }
  state[(size_t)slot * state_stride + e] = M;
}

// out[t, h, :] = raw[t, h, :] / sqrt(mean(raw[t, h, :]^2) + eps) * w; one warp per (token, head).
template <typename T>
__global__ void head_gain_norm_kernel(const float* raw, const float* __restrict__ w, T* out, int rows, int dv, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (row >= rows) return;
  const float* x = raw + (size_t)row * dv;
  float ss = 0.f;
  for (int c = lane; c < dv; c += 32) ss += x[c] * x[c];
  const float denom = sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int c = lane; c < dv; c += 32) out[(size_t)row * dv + c] = from_f<T>(x[c] / denom * w[c]);
}

// rows of the state a thread of the fused kernel keeps, and lanes that share a column: from dk alone
inline int fused_parts(int dk) { return dk <= 32 ? 1 : dk <= 64 ? 2 : 4; }
inline bool scan_can_fuse(int dk, int dv) { return dv * fused_parts(dk) <= (dk > 128 ? 256 : 512); }

template <typename T, typename SOURCE, int R, int PARTS>
int launch_scan_fused(const SOURCE& src, const float* nw, float* state, long state_stride, const int* cu_q, const int* state_slots,
                      void* out, int B, int heads, int dk, int dv, float eps, int num_slots, int* err, cudaStream_t stream) {
  const int gate_row = R * PARTS + 4 * ((R * PARTS) / 32);
  const int threads = (dv * PARTS + 31) / 32 * 32, cols = threads / PARTS;
  const size_t smem = ((size_t)3 * HG_TT * gate_row + 2 * (size_t)HG_TT * cols) * sizeof(float);
  auto kernel = matrix_scan_fused_kernel<T, SOURCE, R, PARTS>;
  if (smem > 48 * 1024) {      // a head of 256 gates: three rows of gates for 16 tokens pass the default limit
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_kernel(kernel, dim3(heads, B), dim3(threads), smem, stream, src, nw, state, state_stride, cu_q, state_slots, (T*)out,
                       heads, dk, dv, eps, num_slots, err);
}

// One token a request: threads by the size of a head, and columns a thread.  dk up to 256 (a gate a thread).
template <typename T, typename SOURCE>
int launch_scan_step(const SOURCE& src, const float* nw, float* state, long state_stride, const int* cu_q, const int* state_slots,
                     void* out, float* raw, int B, int heads, int dk, int dv, float eps, int num_slots, int* err, cudaStream_t stream) {
  const bool vec = dv % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
  const int threads = dk * dv >= 16384 || dv > (vec ? 1024 : 256) ? 512 : 256;
  if (dv > threads * (vec ? 4 : 1) || dk > 256) return VOB_UNSUPPORTED;
  const int groups = threads / (vec ? dv / 4 : dv);
  const size_t smem = ((size_t)3 * dk + (size_t)groups * dv) * sizeof(float);
#define VOB_ST(VV, NN)                                                                                                             \
  return launch_kernel(matrix_scan_step_kernel<T, SOURCE, VV, NN>, dim3(heads, B), dim3(NN), smem, stream, src, nw, state, state_stride, \
                       cu_q, state_slots, (T*)out, raw, heads, dk, dv, eps, num_slots, err)
  if (vec && threads == 512) VOB_ST(4, 512);
  if (vec) VOB_ST(4, 256);
  if (threads == 512) VOB_ST(1, 512);
  VOB_ST(1, 256);
#undef VOB_ST
}
inline bool scan_can_step(int dk, int dv) { return dk <= 256 && dv <= 512; }

inline int tile_parts(int dk) {
  int p = 2;
  while (p * MS_R < dk) p <<= 1;
  return p;
}
// walker threads of a block, and blocks a head
inline int tile_walkers(int dk, int dv) {
  const int per_warp = 32 / tile_parts(dk) * MS_C;
  return min(MS_MAX_WALKERS, (dv + per_warp - 1) / per_warp * 32);
}
inline int tile_col_blocks(int dk, int dv) {
  const int cols = tile_walkers(dk, dv) / tile_parts(dk) * MS_C;
  return (dv + cols - 1) / cols;
}

template <typename SOURCE, int PARTS, bool OUT>
int launch_scan_tile(const SOURCE& src, float* state, long state_stride, const int* cu_q, const int* state_slots, float* raw, float* ends,
                     int B, int chunks, int heads, int dk, int dv, int num_slots, int mode, int* err, cudaStream_t stream) {
  const int walkers = tile_walkers(dk, dv), cols = walkers / PARTS * MS_C, col_blocks = tile_col_blocks(dk, dv);
  const size_t smem = (size_t)2 * HG_TT * ((SOURCE::DECAY == DECAY_ROW ? 3 : 2) * PARTS * MS_R + cols + (SOURCE::DECAY == DECAY_TOKEN ? 1 : 0)) *
                      sizeof(float);
  auto kernel = matrix_scan_tile_kernel<SOURCE, PARTS, OUT>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_kernel(kernel, dim3(heads * col_blocks, B, chunks), dim3(MS_LOADERS + walkers), smem, stream, src, state, state_stride,
                       cu_q, state_slots, raw, ends, heads, dk, dv, col_blocks, num_slots, mode, err);
}

template <typename SOURCE>
int dispatch_scan_tile(int mode, const SOURCE& src, float* state, long state_stride, const int* cu_q, const int* state_slots, float* raw, float* ends,
                       int B, int chunks, int heads, int dk, int dv, int num_slots, int* err, cudaStream_t stream) {
#define VOB_MT(PP)                                                                                                                 \
  case PP:                                                                                                                         \
    if (mode == 1)                                                                                                                 \
      return launch_scan_tile<SOURCE, PP, false>(src, state, state_stride, cu_q, state_slots, raw, ends, B, chunks, heads, dk, dv, \
                                                 num_slots, mode, err, stream);                                                    \
    return launch_scan_tile<SOURCE, PP, true>(src, state, state_stride, cu_q, state_slots, raw, ends, B, chunks, heads, dk, dv,    \
                                              num_slots, mode, err, stream)
  switch (tile_parts(dk)) {
    VOB_MT(2); VOB_MT(4); VOB_MT(8); VOB_MT(16); VOB_MT(32);
  }
#undef VOB_MT
  return VOB_UNSUPPORTED;
}

// The recurrence of any source over a step; with `norm` the head norm that follows an unfused walk.
template <typename T, typename SOURCE>
int run_matrix_scan(const SOURCE& src, const float* nw, float* state, long state_stride, const int* cu_q, const int* state_slots,
                    void* out, float* raw, float* scratch, int Tn, int B, int chunks, int heads, int dk, int dv, float eps,
                    int num_slots, int fuse, int single, int norm, int* err, cudaStream_t stream) {
  const long per = (long)heads * dk * (dv + (SOURCE::NORMALISER ? 1 : 0));
  if (heads <= 0 || dk <= 0 || dv <= 0 || dk > 256 || B > 65535 || (!fuse && !raw) ||
      (fuse && !(single ? scan_can_step(dk, dv) : scan_can_fuse(dk, dv))) || chunks < 1 || chunks > HG_MAX_CHUNKS || (chunks > 1 && (fuse || !scratch)) || state_stride < per + (SOURCE::NORMALISER ? heads : 0))
    return VOB_UNSUPPORTED;
  int code = 0;
  // (a source that makes its head gates itself walks fused only, one whose gates are ready never)
  if constexpr (SOURCE::HEAD_GATES || !SOURCE::NORMALISER) {
    if (single && (fuse || !norm))
      return launch_scan_step<T>(src, nw, state, state_stride, cu_q, state_slots, fuse ? out : nullptr, fuse ? nullptr : raw, B, heads, dk, dv,
                                 eps, num_slots, err, stream);
    if (fuse) {
#define VOB_SF(RR, PP) return launch_scan_fused<T, SOURCE, RR, PP>(src, nw, state, state_stride, cu_q, state_slots, out, B, heads, dk, dv, eps, num_slots, err, stream)
      if (dk <= 16) VOB_SF(16, 1);
      if (dk <= 32) VOB_SF(32, 1);
      if (dk <= 64) VOB_SF(32, 2);
      if (dk <= 128) VOB_SF(32, 4);
      VOB_SF(64, 4);
#undef VOB_SF
    }
  }
  if constexpr (SOURCE::HEAD_GATES) return VOB_UNSUPPORTED;
  else if (chunks <= 1) {
    code = dispatch_scan_tile(0, src, state, state_stride, cu_q, state_slots, raw, nullptr, B, 1, heads, dk, dv, num_slots, err,
                                         stream);
  } else {
    float* ends = scratch;
    float* gates = scratch + (size_t)B * chunks * per;
    code = dispatch_scan_tile(1, src, state, state_stride, cu_q, state_slots, raw, ends, B, chunks, heads, dk, dv, num_slots, err,
                                         stream);
    if (code != 0) return code;
    if constexpr (!SOURCE::NORMALISER) {      // (a source with a normaliser leaves the decays beside it)
      code = launch_kernel(matrix_scan_range_decay_kernel<SOURCE>, dim3((heads * dk + 31) / 32, B, chunks), dim3(256), 0, stream, src,
                           gates, cu_q, heads, dk);
      if (code != 0) return code;
    }
    code = launch_kernel(matrix_scan_join_kernel, dim3((unsigned)((per + 255) / 256), B), dim3(256), 0, stream, state, state_stride, ends,
                         (const float*)gates, cu_q, state_slots, chunks, heads, dk, dv, per, num_slots);
    if (code != 0) return code;
    code = dispatch_scan_tile(2, src, state, state_stride, cu_q, state_slots, raw, ends, B, chunks, heads, dk, dv, num_slots, err,
                                         stream);
  }
  if (code != 0 || !norm) return code;
  const int rows = Tn * heads;
  return launch_kernel(head_gain_norm_kernel<T>, dim3((rows + 3) / 4), dim3(128), 0, stream, (const float*)raw, nw, (T*)out, rows, dv,
                       eps);
}

}  // namespace vob

using namespace vob;

// zxg [T, 3W], bz and bx [W] of the model's type; state float [num_slots, W]; cu_q [B+1]; state_slots [B]; out [T, W].
// `chunks`: 1, 8 or 32 ranges that a request's tokens are cut into (more for longer portions).
VOB_API int vob_mingru_scan(const void* zxg, const void* bz, const void* bx, float* state, const int* cu_q,
                            const int* state_slots, void* out, int B, int W, int num_slots, int chunks, int dtype, int* err,
                            cudaStream_t stream) {
  if (B <= 0 || W <= 0) return 0;
  if (B > 65535 || (chunks != 1 && chunks != 8 && chunks != 32)) return VOB_UNSUPPORTED;
  dim3 grid((W + 31) / 32, B), block(32, chunks);
#define VOB_GRU(TT, NN) \
  return launch_kernel(mingru_scan_kernel<TT, NN>, grid, block, 0, stream, (const TT*)zxg, (const TT*)bz, (const TT*)bx, state, cu_q, \
                       state_slots, (TT*)out, W, num_slots, err)
  if (dtype == VOB_F32) {
    if (chunks == 1) VOB_GRU(float, 1);
    if (chunks == 8) VOB_GRU(float, 8);
    VOB_GRU(float, 32);
  }
  if (dtype == VOB_BF16) {
    if (chunks == 1) VOB_GRU(__nv_bfloat16, 1);
    if (chunks == 8) VOB_GRU(__nv_bfloat16, 8);
    VOB_GRU(__nv_bfloat16, 32);
  }
#undef VOB_GRU
  return VOB_BAD_ARGUMENT;
}

// qfv [T, heads*(2 dk + dv)], bf [heads*dk] of the model's type; lower [heads*dk], nw [dv] float; state float
// [num_slots, heads, dk, dv]; out [T, heads*dv].  `fuse`: one block a (request, head) that also takes the norm (it must
// be able to hold the head: vob_hgrn2_can_fuse); else blocks of 128 threads and raw, float [T, heads*dv], in between.
// `chunks` > 1 (not with fuse): ranges that a request's tokens are cut into, with scratch of
// B * chunks * heads * dk * (dv + 1) floats.
VOB_API int vob_hgrn2_can_fuse(int dk, int dv) { return scan_can_fuse(dk, dv) ? 1 : 0; }

// The same for steps of one token a request (`single` below: no request brings more).
VOB_API int vob_matrix_scan_can_step(int dk, int dv) { return scan_can_step(dk, dv) ? 1 : 0; }

// Ranges that a request's tokens of a step should be cut into (unfused walks): the fewest units of time by a count of float
// instructions a state element (three a token in one walk, five over the two walks of a cut portion, and what the join and the
// launches cost in tokens), given how many blocks fit the device at once.
VOB_API int vob_matrix_scan_chunks(int T, int B, int heads, int dk, int dv) {
  if (B <= 0 || T <= 0 || heads <= 0 || dk <= 0 || dv <= 0) return 1;
  const long blocks = (long)heads * tile_col_blocks(dk, dv) * B, sms = sm_count();
  const double n = (double)T / B;
  int best = 1;
  double least = 3.0 * n * ((blocks + sms - 1) / sms);
  for (int c = 2; c <= HG_MAX_CHUNKS && n / c >= 16; ++c) {
    const double cost = (5.0 * n / c + 120.0) * ((blocks * c + sms - 1) / sms) + 60.0;
    if (cost < least) { least = cost; best = c; }
  }
  return best;
}

VOB_API int vob_hgrn2_scan(const void* qfv, const void* bf, const float* lower, const float* nw, float* state, const int* cu_q,
                           const int* state_slots, void* out, float* raw, float* scratch, int T, int B, int chunks, int heads,
                           int dk, int dv, float eps, int num_slots, int fuse, int single, int dtype, int* err, cudaStream_t stream) {
  if (B <= 0 || T <= 0) return 0;
  const long width = (long)heads * (2 * dk + dv), per = (long)heads * dk * dv;
#define VOB_HS(TT)                                                                                                            \
  return run_matrix_scan<TT>(HgrnSource<TT>{(const TT*)qfv, width, (const TT*)bf, lower, heads, dk, dv}, nw, state, per, cu_q, \
                             state_slots, out, raw, scratch, T, B, chunks, heads, dk, dv, eps, num_slots, fuse, single, 1, err, stream)
  if (dtype == VOB_F32) { VOB_HS(float); }
  if (dtype == VOB_BF16) { VOB_HS(__nv_bfloat16); }
#undef VOB_HS
  return VOB_BAD_ARGUMENT;
}

// rows: `width` elements a token, q | k | v first, the decay's pre-activations (heads*dk) at z_off, the output gate (heads*dv)
// at gate_off; bias float [heads*dk]; nw float [dv]; state float [num_slots, state_stride], the heads' matrices first; out
// [T, heads*dv] of `dtype` with `fuse` (norm and gate included), else raw float [T, heads*dv] and nothing behind it.
VOB_API int vob_gla_scan(const void* rows, long width, int z_off, int gate_off, const float* bias, const float* nw, float* state,
                         long state_stride, const int* cu_q, const int* state_slots, void* out, float* raw, float* scratch, int T,
                         int B, int chunks, int heads, int dk, int dv, float scale, float inv_tau, float eps, int num_slots,
                         int fuse, int single, int dtype, int* err, cudaStream_t stream) {
  if (B <= 0 || T <= 0) return 0;
#define VOB_GS(TT)                                                                                                             \
  return run_matrix_scan<TT>(GlaSource<TT>{(const TT*)rows, width, bias, heads, dk, dv, z_off, gate_off, scale, inv_tau}, nw,  \
                             state, state_stride, cu_q, state_slots, out, raw, scratch, T, B, chunks, heads, dk, dv, eps,      \
                             num_slots, fuse, single, 0, err, stream)
  if (dtype == VOB_F32) { VOB_GS(float); }
  if (dtype == VOB_BF16) { VOB_GS(__nv_bfloat16); }
#undef VOB_GS
  return VOB_BAD_ARGUMENT;
}

// rows: `width` elements a token, q | k | v first; decays float [heads]; raw float [T, heads*dv].
VOB_API int vob_lightning_scan(const void* rows, long width, const float* decays, float* state, long state_stride, const int* cu_q,
                               const int* state_slots, float* raw, float* scratch, int T, int B, int chunks, int heads, int dk,
                               int dv, int num_slots, int single, int dtype, int* err, cudaStream_t stream) {
  if (B <= 0 || T <= 0) return 0;
#define VOB_LS(TT)                                                                                                          \
  return run_matrix_scan<TT>(LightningSource<TT>{(const TT*)rows, width, decays, heads, dk, dv}, (const float*)nullptr,     \
                             state, state_stride, cu_q, state_slots, nullptr, raw, scratch, T, B, chunks, heads, dk, dv, 0.f, \
                             num_slots, 0, single, 0, err, stream)
  if (dtype == VOB_F32) { VOB_LS(float); }
  if (dtype == VOB_BF16) { VOB_LS(__nv_bfloat16); }
#undef VOB_LS
  return VOB_BAD_ARGUMENT;
}

// u and out [T, W] of `dtype`; gates float [T, blocks, 2, W / blocks]; y rows of y_stride elements of `dtype`; br, bi, lam, by
// float [W]; state float [num_slots, state_stride], the W channels first.  `chunks`: 1, 8, 32 or 64 ranges a request's tokens
// are cut into.
VOB_API int vob_lru_scan(const void* u, const float* gates, const void* y, long y_stride, const float* br, const float* bi,
                         const float* lam, const float* by, float* state, long state_stride, const int* cu_q,
                         const int* state_slots, void* out, int B, int W, int blocks, int num_slots, int chunks, int dtype, int* err,
                         cudaStream_t stream) {
  if (B <= 0 || W <= 0) return 0;
  if (B > 65535 || blocks <= 0 || W % blocks || state_stride < W || (chunks != 1 && chunks != 8 && chunks != 32 && chunks != 64)) return VOB_UNSUPPORTED;
#define VOB_LRU(TT, LL, NN)                                                                                                     \
  return launch_kernel(lru_scan_kernel<TT, LL, NN>, dim3((W + LL - 1) / LL, B), dim3(LL, NN), 0, stream, (const TT*)u, gates,   \
                       (const TT*)y, y_stride, br, bi, lam, by, state, state_stride, cu_q, state_slots, (TT*)out, W, W / blocks, \
                       num_slots, err)
#define VOB_LRU_CHUNKS(TT)            \
  do {                                \
    if (chunks == 1) VOB_LRU(TT, 32, 1);   \
    if (chunks == 8) VOB_LRU(TT, 32, 8);   \
    if (chunks == 32) VOB_LRU(TT, 32, 32); \
    VOB_LRU(TT, 16, 64);              \
  } while (0)
  if (dtype == VOB_F32) VOB_LRU_CHUNKS(float);
  if (dtype == VOB_BF16) VOB_LRU_CHUNKS(__nv_bfloat16);
#undef VOB_LRU_CHUNKS
#undef VOB_LRU
  return VOB_BAD_ARGUMENT;
}

// rows: `width` elements a token, q | k | v first, the pre-activations of the input and forget gates (heads each) at i_off and
// f_off, the output gate (heads*dv) at gate_off; bi, bf float [heads]; nw float [heads*dv]; gates float [T, heads, 4]; state float
// [num_slots, state_stride]: the heads' matrices, their normalisers (heads*dk), their running maxima (heads).  With `fuse`, out
// [T, heads*dv] of `dtype`: gates, recurrence, normaliser, head norm, gain and output gate in one launch.  Else raw float
// [T, heads*dv] and nq float [T, heads], and vob_delta_out_norm makes the rest of them and of `gates`.  scratch: B * chunks *
// heads * dk * (dv + 2) floats.
VOB_API int vob_mlstm_scan(const void* rows, long width, int i_off, int f_off, int gate_off, const float* bi, const float* bf,
                           const float* nw, float* gates, float* state, long state_stride, const int* cu_q, const int* state_slots,
                           void* out, float* raw, float* nq, float* scratch, int T, int B, int chunks, int heads, int dk, int dv,
                           float scale, float cap, float eps, int num_slots, int fuse, int single, int dtype, int* err,
                           cudaStream_t stream) {
  if (B <= 0 || T <= 0) return 0;
  if (!(cap > 0.f) || (!fuse && (!nq || !gates || ((uintptr_t)gates & 15)))) return VOB_BAD_ARGUMENT;
  if (heads <= 0 || B > 65535) return VOB_UNSUPPORTED;
#define VOB_ML(TT, GG)                                                                                                          \
  const MlstmSource<TT, GG> src{(const TT*)rows, width, bi, bf, (const float4*)gates, nq, heads, dk, dv, i_off, f_off, gate_off, \
                                scale, cap};                                                                                    \
  if constexpr (GG) {                                                                                                           \
    const int code = launch_kernel(mlstm_gates_kernel<TT>, dim3(heads, B), dim3(MG_NT), 0, stream, src, (float4*)gates, state,  \
                                   state_stride, cu_q, state_slots, num_slots, err);                                            \
    if (code != 0) return code;                                                                                                 \
  }                                                                                                                             \
  return run_matrix_scan<TT>(src, nw, state, state_stride, cu_q, state_slots, out, raw, scratch, T, B, chunks, heads, dk, dv,   \
                             eps, num_slots, fuse, single, 0, err, stream)
  if (dtype == VOB_F32) {
    if (fuse) { VOB_ML(float, false); }
    VOB_ML(float, true);
  }
  if (dtype == VOB_BF16) {
    if (fuse) { VOB_ML(__nv_bfloat16, false); }
    VOB_ML(__nv_bfloat16, true);
  }
#undef VOB_ML
  return VOB_BAD_ARGUMENT;
}
