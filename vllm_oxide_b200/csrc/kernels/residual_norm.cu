// One float residual stream with a norm on both sides of every sublayer ("sandwich" norms):
//
//     x <- x + RMSNorm(y) * w_post          y: the output of the sublayer before (mixer or feed-forward)
//     h  = RMSNorm(x) * w_pre               what the next sublayer reads
//
// One launch does, for every token, any part of that chain in a single pass over the row:
//   (1) x = 0 (`init`: the row begins here, e.g. with the embedded token as y) or x = stream[token];
//   (2) with y:       x += y / sqrt(mean(y^2) + eps) * w_post      (w_post null: x += y)
//   (3) with inject:  x += inject[token]                           (a float row added as it is)
//   (4) x is stored to the stream if (1)-(3) changed it, and to `keep` if given (a second copy that later steps add back);
//   (5) with w_pre:   out = x / sqrt(mean(x^2) + eps) * w_pre.
// With a list of rows, (5) is computed for those source rows only and nothing is stored (the model's last norm on the
// rows whose logits are wanted).
//
// A second kernel, residual_norm_shift_step, is the same chain (without `inject` and `keep`) followed by a token shift, for
// layers whose mixer reads a mix of a token's normed row and the row of the token before it:
//     h_t = RMSNorm(x_t) * w_pre;   out_t = h_t + (h_(t-1) - h_t) * shift          (shift: a number a channel)
// with h_(-1) of a portion from the request's state slot (zeros for a new request), where the portion's last h is left.
// A block walks a few tokens and keeps the last h on chip; the h of the token before its first, and (in the block of a
// portion's first token) the h of the portion's last token, are made again from the rows they come from, so that no block
// waits for another.  For that the new stream goes to a buffer of its own (stream_out) while all blocks read the old one.
//
// The stream, the norms and the sums are float on both paths; y and out are of the model's type T.  A block of fixed
// size takes a row, so the order of additions in a sum of squares depends on the row's width only.
#include "common.cuh"

namespace vob {

constexpr int RN_NT = 256;

template <typename T, int V> struct RowAccess;   // V elements at a time
template <typename T> struct RowAccess<T, 1> {
  static __device__ __forceinline__ void load(const T* p, float (&v)[1]) { v[0] = to_f<T>(p[0]); }
  static __device__ __forceinline__ void store(T* p, const float (&v)[1]) { p[0] = from_f<T>(v[0]); }
};
template <> struct RowAccess<float, 4> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 r = *reinterpret_cast<const float4*>(p);
    v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct RowAccess<__nv_bfloat16, 4> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 r = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
    const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    uint2 r;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&r);
    h[0] = __floats2bfloat162_rn(v[0], v[1]);
    h[1] = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = r;
  }
};

template <typename T, int V>
__global__ void __launch_bounds__(RN_NT)
residual_norm_step_kernel(float* stream, const T* y, const float* __restrict__ w_post, const float* inject, float* keep,
                          const float* __restrict__ w_pre, T* out, const int* __restrict__ rows, int num_src_rows, int D,
                          float eps, int init, int* err) {
  extern __shared__ float4 rn_smem4[];
  float* xrow = reinterpret_cast<float*>(rn_smem4);   // [D] the new row
  float* yrow = xrow + D;                              // [D] the sublayer's output (only with y)
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  int src = r;
  if (rows) {
    src = rows[r];
    if (src < 0 || src >= num_src_rows) {
      if (threadIdx.x == 0) atomicOr(err, VOB_ERR_ROW);
      return;
    }
  }
  const size_t base = (size_t)src * D;
  float inv_y = 1.f;
  if (y) {
    float ss = 0.f;
    for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
      float v[V];
      RowAccess<T, V>::load(y + base + d, v);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        yrow[d + j] = v[j];
        ss = fmaf(v[j], v[j], ss);
      }
    }
    const float total = block_sum<RN_NT>(ss, scratch);
    if (w_post) inv_y = 1.f / sqrtf(total / (float)D + eps);
  }
  const bool changed = init || y || inject;
  const bool store = rows == nullptr;
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
    float x[V];
    if (init) {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] = 0.f;
    } else {
      RowAccess<float, V>::load(stream + base + d, x);
    }
    if (y) {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += w_post ? yrow[d + j] * inv_y * w_post[d + j] : yrow[d + j];
    }
    if (inject) {
      float e[V];
      RowAccess<float, V>::load(inject + base + d, e);
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += e[j];
    }
    if (store && changed) RowAccess<float, V>::store(stream + base + d, x);
    if (store && keep) RowAccess<float, V>::store(keep + base + d, x);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      xrow[d + j] = x[j];
      ss = fmaf(x[j], x[j], ss);
    }
  }
  if (!out) return;
  const float total = block_sum<RN_NT>(ss, scratch);
  const float inv_x = 1.f / sqrtf(total / (float)D + eps);
  for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
    float o[V];
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = xrow[d + j] * inv_x * (w_pre ? w_pre[d + j] : 1.f);
    RowAccess<T, V>::store(out + (size_t)r * D + d, o);
  }
}

// ---- rows in registers: widths that are a multiple of 4 and fit NV groups of 4 elements a thread.  All loads of a row are issued
// before its first sum, and (in a walk) the next row's before this row's sums, so a block waits for memory once a row.  The same
// arithmetic as the kernels that keep the row in shared memory.
template <typename T, int NT, int NV>
struct StreamRow {
  float x[NV][4];      // the stream's row
  float y[NV][4];      // the sublayer's output
  __device__ __forceinline__ void load(const float* stream, const T* yin, size_t base, int D, bool init) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
#pragma unroll
      for (int j = 0; j < 4; ++j) x[i][j] = y[i][j] = 0.f;
      if (d < D) {
        if (!init) RowAccess<float, 4>::load(stream + base + d, x[i]);
        if (yin) RowAccess<T, 4>::load(yin + base + d, y[i]);
      }
    }
  }
  // x += RMSNorm(y) * w_post (w_post null: x += y; no y: nothing)
  __device__ __forceinline__ void add(bool has_y, const float* __restrict__ w_post, int D, float eps, float* scratch) {
    if (!has_y) return;
    float inv = 1.f;
    if (w_post) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) ss = fmaf(y[i][j], y[i][j], ss);
      inv = 1.f / sqrtf(block_sum<NT>(ss, scratch) / (float)D + eps);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
      if (d < D) {
        float w[4] = {1.f, 1.f, 1.f, 1.f};
        if (w_post) RowAccess<float, 4>::load(w_post + d, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[i][j] += w_post ? y[i][j] * inv * w[j] : y[i][j];
      }
    }
  }
  __device__ __forceinline__ float inv_rms(int D, float eps, float* scratch) const {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) ss = fmaf(x[i][j], x[i][j], ss);
    return 1.f / sqrtf(block_sum<NT>(ss, scratch) / (float)D + eps);
  }
  // x / rms * w_pre into h
  __device__ __forceinline__ void normed(float inv, const float* __restrict__ w_pre, int D, float (&h)[NV][4]) const {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
      float w[4] = {1.f, 1.f, 1.f, 1.f};
      if (w_pre && d < D) RowAccess<float, 4>::load(w_pre + d, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) h[i][j] = x[i][j] * inv * w[j];
    }
  }
  template <typename TO>
  static __device__ __forceinline__ void put(TO* p, const float (&v)[NV][4], int D) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
      if (d < D) RowAccess<TO, 4>::store(p + d, v[i]);
    }
  }
};

template <typename T, int NT, int NV>
__global__ void __launch_bounds__(NT)
residual_norm_step_regs_kernel(float* stream, const T* y, const float* __restrict__ w_post, const float* inject, float* keep,
                               const float* __restrict__ w_pre, T* out, const int* __restrict__ rows, int num_src_rows, int D,
                               float eps, int init, int* err) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x;
  int src = r;
  if (rows) {
    src = rows[r];
    if (src < 0 || src >= num_src_rows) {
      if (threadIdx.x == 0) atomicOr(err, VOB_ERR_ROW);
      return;
    }
  }
  const size_t base = (size_t)src * D;
  StreamRow<T, NT, NV> row;
  row.load(stream, y, base, D, init != 0);
  row.add(y != nullptr, w_post, D, eps, scratch);
  if (inject) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
      if (d < D) {
        float e[4];
        RowAccess<float, 4>::load(inject + base + d, e);
#pragma unroll
        for (int j = 0; j < 4; ++j) row.x[i][j] += e[j];
      }
    }
  }
  if (!rows) {
    if (init || y || inject) row.put(stream + base, row.x, D);
    if (keep) row.put(keep + base, row.x, D);
  }
  if (!out) return;
  float h[NV][4];
  row.normed(row.inv_rms(D, eps, scratch), w_pre, D, h);
  row.put(out + (size_t)r * D, h, D);
}

template <typename T, int NT, int NV>
__global__ void __launch_bounds__(NT)
residual_norm_shift_regs_kernel(const float* stream, float* stream_out, const T* y, const float* __restrict__ w_post,
                                const float* __restrict__ w_pre, const float* __restrict__ shift, float* state, long state_stride,
                                const int* __restrict__ token_req, const int* __restrict__ cu_q, const int* __restrict__ state_slots,
                                T* out, int num_tokens, int walk, int D, float eps, long num_slots, int* err) {
  using Row = StreamRow<T, NT, NV>;
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int t0 = blockIdx.x * walk, t1 = min(num_tokens, t0 + walk);
  int req = token_req[t0];
  const bool ahead = req >= 0 && t0 > cu_q[req];        // the first token has one before it in its portion
  pdl_wait();
  float before[NV][4], h[NV][4];
  Row next, row;
  if (ahead) row.load(stream, y, (size_t)(t0 - 1) * D, D, false);
  next.load(stream, y, (size_t)t0 * D, D, false);
  if (ahead) {
    row.add(y != nullptr, w_post, D, eps, scratch);
    row.normed(row.inv_rms(D, eps, scratch), w_pre, D, before);
  }
  for (int t = t0; t < t1; ++t) {
    row = next;
    if (t + 1 < t1) next.load(stream, y, (size_t)(t + 1) * D, D, false);
    req = token_req[t];
    int slot = -1, first = t, last = t;
    if (req >= 0) {
      slot = state_slots[req];
      first = cu_q[req];
      last = cu_q[req + 1] - 1;
      if (slot < 0 || slot >= num_slots) {
        if (threadIdx.x == 0) atomicOr(err, VOB_ERR_SLOT);
        slot = -1;
      }
    }
    float* kept = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
    if (t == first) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = (i * NT + threadIdx.x) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j) before[i][j] = kept && d < D ? kept[d + j] : 0.f;
      }
    }
    row.add(y != nullptr, w_post, D, eps, scratch);
    if (y) Row::put(stream_out + (size_t)t * D, row.x, D);
    row.normed(row.inv_rms(D, eps, scratch), w_pre, D, h);
    if (kept && t == last && t == first) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = (i * NT + threadIdx.x) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (d < D) kept[d + j] = h[i][j];
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int d = (i * NT + threadIdx.x) * 4;
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      if (req >= 0 && d < D) RowAccess<float, 4>::load(shift + d, s);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float mixed = fmaf(before[i][j] - h[i][j], s[j], h[i][j]);
        before[i][j] = h[i][j];
        h[i][j] = req >= 0 ? mixed : h[i][j];
      }
    }
    Row::put(out + (size_t)t * D, h, D);
    if (kept && t == first && last > first) {
      // the portion's last h into the slot: by the block that has just read the slot, so that nothing is overwritten early
      row.load(stream, y, (size_t)last * D, D, false);
      row.add(y != nullptr, w_post, D, eps, scratch);
      row.normed(row.inv_rms(D, eps, scratch), w_pre, D, h);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int d = (i * NT + threadIdx.x) * 4;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (d < D) kept[d + j] = h[i][j];
      }
    }
  }
}

// The normed row of token t, left in `row` as x (the caller multiplies by the returned 1 / rms); with `put` the new stream
// row is stored.
template <typename T, int V>
__device__ __forceinline__ float shift_row(const float* stream, float* stream_out, const T* y, const float* __restrict__ w_post,
                                           float* row, int t, bool put, int D, float eps, float* scratch) {
  const size_t base = (size_t)t * D;
  float inv_y = 1.f;
  if (y) {
    float ss = 0.f;
    for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
      float v[V];
      RowAccess<T, V>::load(y + base + d, v);
#pragma unroll
      for (int j = 0; j < V; ++j) { row[d + j] = v[j]; ss = fmaf(v[j], v[j], ss); }
    }
    if (w_post) inv_y = 1.f / sqrtf(block_sum<RN_NT>(ss, scratch) / (float)D + eps);
  }
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
    float x[V];
    RowAccess<float, V>::load(stream + base + d, x);
    if (y) {
#pragma unroll
      for (int j = 0; j < V; ++j) x[j] += w_post ? row[d + j] * inv_y * w_post[d + j] : row[d + j];
      if (put) RowAccess<float, V>::store(stream_out + base + d, x);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) { row[d + j] = x[j]; ss = fmaf(x[j], x[j], ss); }
  }
  return 1.f / sqrtf(block_sum<RN_NT>(ss, scratch) / (float)D + eps);
}

template <typename T, int V>
__global__ void __launch_bounds__(RN_NT)
residual_norm_shift_kernel(const float* stream, float* stream_out, const T* y, const float* __restrict__ w_post,
                           const float* __restrict__ w_pre, const float* __restrict__ shift, float* state, long state_stride,
                           const int* __restrict__ token_req, const int* __restrict__ cu_q, const int* __restrict__ state_slots,
                           T* out, int num_tokens, int walk, int D, float eps, long num_slots, int* err) {
  extern __shared__ float4 rn_smem4[];
  float* row = reinterpret_cast<float*>(rn_smem4);    // [D] the token's stream row
  float* before = row + D;                             // [D] h of the token before
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  bool have = false;                                   // `before` is that of the token at hand
  for (int k = 0; k < walk; ++k) {
    const int t = blockIdx.x * walk + k;
    if (t >= num_tokens) break;
    const int req = token_req[t];
    int slot = -1, first = t, last = t;
    if (req >= 0) {
      slot = state_slots[req];
      first = cu_q[req];
      last = cu_q[req + 1] - 1;
      if (slot < 0 || slot >= num_slots) {
        if (threadIdx.x == 0) atomicOr(err, VOB_ERR_SLOT);
        slot = -1;
      }
    }
    float* kept = slot >= 0 ? state + (size_t)slot * state_stride : nullptr;
    // (a thread reads and writes the same elements of `row` and `before` in every pass)
    if (t == first) {
      for (int d = threadIdx.x * V; d < D; d += RN_NT * V)
#pragma unroll
        for (int j = 0; j < V; ++j) before[d + j] = kept ? kept[d + j] : 0.f;
    } else if (!have) {
      const float inv = shift_row<T, V>(stream, stream_out, y, w_post, row, t - 1, false, D, eps, scratch);
      for (int d = threadIdx.x * V; d < D; d += RN_NT * V)
#pragma unroll
        for (int j = 0; j < V; ++j) before[d + j] = row[d + j] * inv * w_pre[d + j];
    }
    const float inv = shift_row<T, V>(stream, stream_out, y, w_post, row, t, true, D, eps, scratch);
    for (int d = threadIdx.x * V; d < D; d += RN_NT * V) {
      float o[V];
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float h = row[d + j] * inv * w_pre[d + j];
        o[j] = req >= 0 ? fmaf(before[d + j] - h, shift[d + j], h) : h;
        before[d + j] = h;
        if (kept && t == last && t == first) kept[d + j] = h;
      }
      RowAccess<T, V>::store(out + (size_t)t * D + d, o);
    }
    have = true;
    if (kept && t == first && last > first) {
      // the portion's last h into the slot: by the block that has just read the slot, so that nothing is overwritten early
      const float inv_last = shift_row<T, V>(stream, stream_out, y, w_post, row, last, false, D, eps, scratch);
      for (int d = threadIdx.x * V; d < D; d += RN_NT * V)
#pragma unroll
        for (int j = 0; j < V; ++j) kept[d + j] = row[d + j] * inv_last * w_pre[d + j];
    }
  }
}

}  // namespace vob

using namespace vob;

// stream [num_src_rows, D] float; y [num_src_rows, D] and out [n_out, D] of `dtype`; w_post, w_pre [D] float; inject and
// keep [num_src_rows, D] float; rows [n_out] source rows or null (then n_out == num_src_rows).  Any of y, w_post, inject,
// keep, w_pre / out may be null.
VOB_API int vob_residual_norm_step(float* stream, const void* y, const float* w_post, const float* inject, float* keep,
                                   const float* w_pre, void* out, const int* rows, int n_out, int num_src_rows, int D,
                                   float eps, int init, int dtype, int* err, cudaStream_t stream_) {
  if (n_out <= 0) return 0;
  if (D <= 0 || (rows && (keep || !out))) return VOB_BAD_ARGUMENT;
  const size_t smem = (size_t)2 * D * sizeof(float);
  if (smem > 200 * 1024) return VOB_UNSUPPORTED;
  const bool vec = D % 4 == 0 && (((uintptr_t)stream | (uintptr_t)y | (uintptr_t)inject | (uintptr_t)keep | (uintptr_t)out |
                                    (uintptr_t)w_post | (uintptr_t)w_pre) % 16) == 0;
#define VOB_RN_REGS(TYPE, NT, NV)                                                                                           \
  return launch_kernel(residual_norm_step_regs_kernel<TYPE, NT, NV>, dim3(n_out), NT, 0, stream_, stream, (const TYPE*)y, w_post, \
                       inject, keep, w_pre, (TYPE*)out, rows, num_src_rows, D, eps, init, err)
#define VOB_RN_WIDTHS(TYPE)                    \
  do {                                         \
    if (D <= 512) VOB_RN_REGS(TYPE, 128, 1);   \
    if (D <= 1024) VOB_RN_REGS(TYPE, 256, 1);  \
    if (D <= 2048) VOB_RN_REGS(TYPE, 256, 2);  \
    if (D <= 4096) VOB_RN_REGS(TYPE, 256, 4);  \
    VOB_RN_REGS(TYPE, 512, 4);                 \
  } while (0)
  if (vec && D <= 8192) {
    if (dtype == VOB_F32) VOB_RN_WIDTHS(float);
    if (dtype == VOB_BF16) VOB_RN_WIDTHS(__nv_bfloat16);
  }
#undef VOB_RN_WIDTHS
#undef VOB_RN_REGS
#define VOB_RN_LAUNCH(TYPE, V)                                                                                            \
  do {                                                                                                                    \
    if (smem > 48 * 1024)                                                                                                 \
      cudaFuncSetAttribute(residual_norm_step_kernel<TYPE, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    return launch_kernel(residual_norm_step_kernel<TYPE, V>, dim3(n_out), RN_NT, smem, stream_, stream, (const TYPE*)y,   \
                         w_post, inject, keep, w_pre, (TYPE*)out, rows, num_src_rows, D, eps, init, err);                 \
  } while (0)
  if (dtype == VOB_F32) {
    if (vec) VOB_RN_LAUNCH(float, 4);
    VOB_RN_LAUNCH(float, 1);
  }
  if (dtype == VOB_BF16) {
    if (vec) VOB_RN_LAUNCH(__nv_bfloat16, 4);
    VOB_RN_LAUNCH(__nv_bfloat16, 1);
  }
#undef VOB_RN_LAUNCH
  return VOB_BAD_ARGUMENT;
}

// stream [T, D] float, as the sublayer before found it; y [T, D] of `dtype` (null: the stream does not change and stream_out is
// not written) and w_post as above; stream_out [T, D] float, another buffer than `stream`; w_pre, shift [D] float; state float
// [num_slots, state_stride]: the last h of every request, D numbers; out [T, D] of `dtype`.
VOB_API int vob_residual_norm_shift_step(const float* stream, float* stream_out, const void* y, const float* w_post, const float* w_pre,
                                         const float* shift, float* state, long state_stride, const int* token_req,
                                         const int* cu_q, const int* state_slots, void* out, int T, int D, float eps,
                                         long num_slots, int dtype, int* err, cudaStream_t stream_) {
  if (T <= 0) return 0;
  if (D <= 0 || !w_pre || !shift || !state || !out || state_stride < D || (y && (!stream_out || stream_out == stream)))
    return VOB_BAD_ARGUMENT;
  const size_t smem = (size_t)2 * D * sizeof(float);
  if (smem > 200 * 1024) return VOB_UNSUPPORTED;
  const bool vec = D % 4 == 0 && (((uintptr_t)stream | (uintptr_t)stream_out | (uintptr_t)y | (uintptr_t)out) % 16) == 0;
  const bool regs = vec && D <= 8192 && (((uintptr_t)w_post | (uintptr_t)w_pre | (uintptr_t)shift) % 16) == 0;
  // a block makes one row more than it walks: few tokens a block while they fill the device, up to eight beyond
  const int walk = max(1, min(8, T / (4 * sm_count())));
#define VOB_RS_REGS(TYPE, NT, NV)                                                                                           \
  return launch_kernel(residual_norm_shift_regs_kernel<TYPE, NT, NV>, dim3((T + walk - 1) / walk), NT, 0, stream_, stream,  \
                       stream_out, (const TYPE*)y, w_post, w_pre, shift, state, state_stride, token_req, cu_q, state_slots, \
                       (TYPE*)out, T, walk, D, eps, num_slots, err)
#define VOB_RS_WIDTHS(TYPE)                    \
  do {                                         \
    if (D <= 512) VOB_RS_REGS(TYPE, 128, 1);   \
    if (D <= 1024) VOB_RS_REGS(TYPE, 256, 1);  \
    if (D <= 2048) VOB_RS_REGS(TYPE, 256, 2);  \
    if (D <= 4096) VOB_RS_REGS(TYPE, 256, 4);  \
    VOB_RS_REGS(TYPE, 512, 4);                 \
  } while (0)
  if (regs) {
    if (dtype == VOB_F32) VOB_RS_WIDTHS(float);
    if (dtype == VOB_BF16) VOB_RS_WIDTHS(__nv_bfloat16);
  }
#undef VOB_RS_WIDTHS
#undef VOB_RS_REGS
#define VOB_RS_LAUNCH(TYPE, V)                                                                                             \
  do {                                                                                                                     \
    if (smem > 48 * 1024)                                                                                                  \
      cudaFuncSetAttribute(residual_norm_shift_kernel<TYPE, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);   \
    return launch_kernel(residual_norm_shift_kernel<TYPE, V>, dim3((T + walk - 1) / walk), RN_NT, smem, stream_, stream,   \
                         stream_out, (const TYPE*)y, w_post, w_pre, shift, state, state_stride, token_req, cu_q,           \
                         state_slots, (TYPE*)out, T, walk, D, eps, num_slots, err);                                        \
  } while (0)
  if (dtype == VOB_F32) {
    if (vec) VOB_RS_LAUNCH(float, 4);
    VOB_RS_LAUNCH(float, 1);
  }
  if (dtype == VOB_BF16) {
    if (vec) VOB_RS_LAUNCH(__nv_bfloat16, 4);
    VOB_RS_LAUNCH(__nv_bfloat16, 1);
  }
#undef VOB_RS_LAUNCH
  return VOB_BAD_ARGUMENT;
}
