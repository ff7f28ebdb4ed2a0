// Building blocks of the bfloat16 attention kernels: m16n8k16 tensor-core products on a 16-row
// query tile, ldmatrix loads from padded shared-memory rows, cp.async copies of cache rows, and the
// online softmax in float (base-2 exponentials; scores are pre-multiplied by log2(e)).
//
// The head size is a compile-time constant: the file that includes this header is compiled once
// per head size with -DVOB_HD=<multiple of 16, at most 256>.
#pragma once
#include "tensor_map.cuh"

#ifndef VOB_HD
#define VOB_HD 128
#endif

namespace vob {

constexpr int HD = VOB_HD;
static_assert(HD % 16 == 0 && HD >= 16 && HD <= 256, "head size must be a multiple of 16 up to 256");
constexpr int ROW_BYTES = HD * 2 + 16;  // one key or value row in shared memory, padded against bank conflicts
constexpr int KSTEPS = HD / 16;         // k-steps of a Q.K^T product
constexpr int DTILES = HD / 8;          // 8-wide output tiles of a P.V product
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  const int bytes = valid ? 16 : 0;  // 0: nothing is read, 16 zero bytes are written
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], const void* smem_row) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem_row);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem_row) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem_row);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}

// d[16x8] += a[16x16] * b[16x8], bfloat16 in, float accumulate
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// 2^x by the hardware approximation (2 ulp; -inf gives 0): the softmax needs no more on the bfloat16 path.
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

// 1 / x by the hardware approximation (1 ulp; +inf gives 0).
__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

// What a head's softmax does besides scaling and the causal mask, and what may come after it.  `sink`: the softmax has a
// silent extra entry of score 0 that has no value; it adds 2^(0 - M) to a denominator that is taken relative to M (scores in
// the base-2 domain).  `sinks` (float [heads]): the extra entry's score is a number of the head's own instead, as it is (the
// scale does not touch it).  `gate`: head h of token t is multiplied by sigmoid(gate[t * gate_stride + h]).  `cap_out` > 0: a
// score becomes cap * tanh(score / cap); the two factors are cap_in = scale / cap * 2 log2(e) (on the raw product) and
// cap_out = cap * log2(e) (see head_options).  `chunk` > 0: a query sees only the keys of its own block of `chunk`
// positions, counted from position 0.  `value_div` > 1: the value plane has kv_heads / value_div heads, and key head k
// reads value head k / value_div (key heads that are several maps over one value head).  `out_float`: the output is float
// (same shape), for heads that are combined before anything rounds them.  All zero leaves the softmax as it is.
struct HeadEpilogue {
  int sink;
  const float* sinks;
  const __nv_bfloat16* gate;
  long gate_stride;
  float cap_in, cap_out;
  int chunk;
  int value_div;
  int out_float;
  int keep_first;             // > 0: the keys at positions below it are seen by every later query, whatever the window
  const float* dist_bias;     // [heads, dist_rows] float or null: entry min(query position - key position, dist_rows - 1) of
  int dist_rows;              // the head's row is added to the scaled score (a learned bias by distance; neighbouring keys
                              // read neighbouring floats)
};
__host__ inline HeadEpilogue head_options(int sink, const float* sinks, const void* gate, long gate_stride, float softcap, float scale, int chunk,
                                          int value_div, int out_float = 0, int keep_first = 0, const float* dist_bias = nullptr,
                                          int dist_rows = 0) {
  HeadEpilogue ep{sink, sinks, (const __nv_bfloat16*)gate, gate_stride, 0.f, 0.f, chunk > 0 ? chunk : 0, value_div > 1 ? value_div : 1,
                  out_float, keep_first > 0 ? keep_first : 0, dist_rows > 0 ? dist_bias : nullptr, dist_rows};
  if (softcap > 0.f) {
    ep.cap_in = scale / softcap * 2.f * 1.4426950408889634f;
    ep.cap_out = softcap * 1.4426950408889634f;
  }
  return ep;
}
// The first key that the query at `pos` sees.  It does not fall as `pos` grows.
__device__ __forceinline__ int first_key(int pos, int window, const HeadEpilogue& ep) {
  if (ep.chunk > 0) return pos / ep.chunk * ep.chunk;
  return window > 0 ? max(0, pos - window + 1) : 0;
}
// A raw product as a score in the base-2 domain: raw * sc (sc = scale * log2(e)), capped if the head caps its scores:
// cap * tanh(x) * log2(e) with tanh(x) = 1 - 2 / (1 + e^(2x)), which the hardware's 2^x and division give to a few ulp of 1
// (the tanh approximation of the hardware is good to 2^-11 only, which a cap of 30 would turn into 1% of a weight).
__device__ __forceinline__ float score2(float raw, float sc, const HeadEpilogue& ep) {
  if (ep.cap_out > 0.f) {
    return fmaf(-2.f * ep.cap_out, fast_rcp(1.f + fast_exp2(raw * ep.cap_in)), ep.cap_out);
  }
  return raw * sc;
}
// The bias by distance of head `head` (of `nh`) for a key `dist` positions behind its query, in the base-2 domain.
__device__ __forceinline__ float dist_term(const HeadEpilogue& ep, int dist, int head, int nh) {
  return ep.dist_bias ? ep.dist_bias[(size_t)min(head, nh - 1) * ep.dist_rows + min(dist, ep.dist_rows - 1)] * LOG2E : 0.f;
}
// The same through a head's row of the table, found once (null: no bias).
__device__ __forceinline__ const float* dist_row(const HeadEpilogue& ep, int head, int nh) {
  return ep.dist_bias ? ep.dist_bias + (size_t)min(head, nh - 1) * ep.dist_rows : nullptr;
}
__device__ __forceinline__ float dist_term(const float* row, int dist, int last) { return row ? row[min(dist, last)] * LOG2E : 0.f; }
// Kept first keys beside a window: a kernel that walks ONE range of keys walks a virtual one, the kept keys [0, kept) rounded
// up to whole tiles and, right behind them, the window's keys; `real()` turns a virtual key into its position.  With nothing
// kept, or where the two ranges meet, virtual and real keys are the same.
struct KeptKeys {
  int kept;     // virtual keys below it are positions as they are (0: nothing is mapped)
  int gap;      // virtual keys from `kept` on lie `gap` positions further
  __device__ __forceinline__ int real(int v) const { return (kept > 0 && v >= kept) ? v + gap : v; }
};
// `keep`: kept first keys that lie below the window's first key; `window_start`: where the window's tiles begin (a multiple
// of the copies' granularity, at most the first key).  Returns the map and moves `window_start` to the first virtual key.
__device__ __forceinline__ KeptKeys kept_keys(int keep, int tile, int& window_start) {
  KeptKeys m{0, 0};
  if (keep <= 0) return m;
  const int rounded = (keep + tile - 1) / tile * tile;
  if (rounded >= window_start) { window_start = 0; return m; }      // the two ranges meet: one range from position 0
  m.kept = rounded;
  m.gap = window_start - rounded;
  window_start = 0;
  return m;
}
// Element i of the output.
__device__ __forceinline__ void store_out(__nv_bfloat16* out, size_t i, float v, const HeadEpilogue& ep) {
  if (ep.out_float) reinterpret_cast<float*>(out)[i] = v;
  else out[i] = __float2bfloat16_rn(v);
}
// The value plane's heads and the value head of key head `kh`.
__device__ __forceinline__ int value_heads(int kvh, const HeadEpilogue& ep) { return ep.value_div > 1 ? kvh / ep.value_div : kvh; }
__device__ __forceinline__ int value_head(int kh, const HeadEpilogue& ep) { return ep.value_div > 1 ? kh / ep.value_div : kh; }
// The sink's share of a denominator relative to M.  A maximum far below zero gives +inf, and the head's output 0: the limit.
__device__ __forceinline__ float sink_weight(const HeadEpilogue& ep, float M, int head) {
  if (ep.sinks) return exp2f(fmaf(ep.sinks[head], LOG2E, -M));
  return ep.sink ? exp2f(-M) : 0.f;
}
__device__ __forceinline__ float head_gate(const HeadEpilogue& ep, int t, int head) {
  if (!ep.gate) return 1.f;
  const float g = __bfloat162float(ep.gate[(size_t)t * ep.gate_stride + head]);
  return 1.f / (1.f + __expf(-g));
}

// The largest of three (one instruction on this architecture).
__device__ __forceinline__ float max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;\n" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}

// One warp's state for a 16-row query tile: the thread owns rows g = lane/4 and g+8.
struct WarpSoftmax {
  float m[2] = {-INFINITY, -INFINITY};  // running maximum (base-2 score domain)
  float l[2] = {0.f, 0.f};              // this thread's part of the running sum
  float o[DTILES][4];                   // weighted value sums: o[j] = (row g: d 8j+2t, +1; row g+8: same)
  __device__ __forceinline__ void clear() {
#pragma unroll
    for (int j = 0; j < DTILES; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  }
};

// Scores of the warp's 16 rows against 16 keys whose rows start at `krows` (shared memory):
// s[0] covers keys 0..7, s[1] keys 8..15; thread holds (row g, keys 2t, 2t+1) and (row g+8, same).
__device__ __forceinline__ void qk_16keys(const uint32_t (&q)[KSTEPS][4], const char* krows, int lane, float (&s)[2][4]) {
#pragma unroll
  for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
  const int mi = lane >> 3, r = lane & 7;
  const char* base = krows + ((mi >> 1) * 8 + r) * ROW_BYTES + (mi & 1) * 16;
#pragma unroll
  for (int ks = 0; ks < KSTEPS; ++ks) {
    uint32_t b[4];
    ldmatrix_x4(b, base + ks * 32);
    mma_bf16(s[0], q[ks], b[0], b[1]);
    mma_bf16(s[1], q[ks], b[2], b[3]);
  }
}

// Online-softmax update with the 16 scores per row in s (already scaled to base 2; masked = -inf),
// then o += p * V for the 16 values whose rows start at `vrows`.
__device__ __forceinline__ void softmax_pv_16keys(WarpSoftmax& st, float (&s)[2][4], const char* vrows, int lane) {
  float mx[2];
  mx[0] = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1]));
  mx[1] = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
  }
  float corr[2], mnew[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    mnew[h] = fmaxf(st.m[h], mx[h]);
    corr[h] = (st.m[h] == -INFINITY) ? 0.f : fast_exp2(st.m[h] - mnew[h]);
    st.m[h] = mnew[h];
  }
  float p[2][4];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    // a row that has seen no key yet (maximum -inf) gets a finite stand-in, so that -inf - -inf never occurs
    const float m0 = mnew[0] == -INFINITY ? 0.f : mnew[0], m1 = mnew[1] == -INFINITY ? 0.f : mnew[1];
    p[i][0] = fast_exp2(s[i][0] - m0);
    p[i][1] = fast_exp2(s[i][1] - m0);
    p[i][2] = fast_exp2(s[i][2] - m1);
    p[i][3] = fast_exp2(s[i][3] - m1);
  }
  st.l[0] = st.l[0] * corr[0] + (p[0][0] + p[0][1] + p[1][0] + p[1][1]);
  st.l[1] = st.l[1] * corr[1] + (p[0][2] + p[0][3] + p[1][2] + p[1][3]);
  uint32_t a[4];
  a[0] = pack_bf16(p[0][0], p[0][1]);
  a[1] = pack_bf16(p[0][2], p[0][3]);
  a[2] = pack_bf16(p[1][0], p[1][1]);
  a[3] = pack_bf16(p[1][2], p[1][3]);
  const int mi = lane >> 3, r = lane & 7;
  const char* base = vrows + ((mi & 1) * 8 + r) * ROW_BYTES + (mi >> 1) * 16;
#pragma unroll
  for (int j = 0; j < DTILES; j += 2) {
    st.o[j][0] *= corr[0]; st.o[j][1] *= corr[0]; st.o[j][2] *= corr[1]; st.o[j][3] *= corr[1];
    st.o[j + 1][0] *= corr[0]; st.o[j + 1][1] *= corr[0]; st.o[j + 1][2] *= corr[1]; st.o[j + 1][3] *= corr[1];
    uint32_t b[4];
    ldmatrix_x4_trans(b, base + j * 16);
    mma_bf16(st.o[j], a, b[0], b[1]);
    mma_bf16(st.o[j + 1], a, b[2], b[3]);
  }
}

// The cache rows of a tile are copied in runs of 16 keys.  The caches are [pages, kv_heads, block_size, HD],
// pages hold a multiple of 16 keys and tiles start at multiples of 16, so a run lies in one page and is ONE
// contiguous piece of memory for a head.  Looking the pages up is a global load with a long latency, so it is
// done one tile ahead of the copies that need it (tile_pages), into registers.
constexpr int RUN_KEYS = 16;
constexpr int PAGE_NONE = -2;      // no key of the run is wanted: nothing is looked up, zeros are written

template <int TILE>
__device__ __forceinline__ void tile_pages(int (&pages)[TILE / RUN_KEYS], const int* __restrict__ table, int block_size,
                                           int tile_start, int begin, int end, int keep_end = 0) {
#pragma unroll
  for (int run = 0; run < TILE / RUN_KEYS; ++run) {
    const int key0 = tile_start + run * RUN_KEYS;
    pages[run] = ((key0 < end && key0 + RUN_KEYS > begin) || key0 < keep_end) ? table[key0 / block_size] : PAGE_NONE;
  }
}

// Copies TILE cache rows (keys tile_start .. tile_start+TILE-1 of key/value head kh) into shared memory: K rows
// first, V rows after them; `pages` comes from tile_pages for the same tile.  Keys outside [begin, end) and not below
// `keep_end` are zero-filled (a window group has given the pages below its window back, but for those of kept first keys).
template <int TILE, int THREADS>
__device__ __forceinline__ void load_kv_tile(char* stage, const __nv_bfloat16* kcache,
                                             const __nv_bfloat16* vcache, const int (&pages)[TILE / RUN_KEYS],
                                             int block_size, int kvh, int kh, int tile_start, int begin, int end,
                                             long num_pages, int* err, int v_kvh, int v_kh, int keep_end = 0) {
  constexpr int CHUNKS = HD / 8;                       // 16-byte chunks per row
  constexpr int RUN_CHUNKS = RUN_KEYS * CHUNKS;
  const long head_off = (long)kh * block_size * HD;
  const long page_elems = (long)kvh * block_size * HD;
#pragma unroll
  for (int run = 0; run < TILE / RUN_KEYS; ++run) {
    const int key0 = tile_start + run * RUN_KEYS;
    const int page = pages[run];
    const bool page_ok = page >= 0 && page < num_pages;
    if (!page_ok && page != PAGE_NONE) atomicOr(err, VOB_ERR_PAGE);
    const long base = page_ok ? (long)page * page_elems + head_off + (long)(key0 % block_size) * HD : 0;
    const __nv_bfloat16* ksrc = kcache + base;
    const __nv_bfloat16* vsrc = vcache + (page_ok ? ((long)page * v_kvh + v_kh) * block_size * HD + (long)(key0 % block_size) * HD : 0);
    char* kdst = stage + run * RUN_KEYS * ROW_BYTES;
#pragma unroll
    for (int c = threadIdx.x; c < RUN_CHUNKS; c += THREADS) {
      const int row = c / CHUNKS, col = c - row * CHUNKS;
      const int key = key0 + row;
      const bool valid = page_ok && ((key >= begin && key < end) || key < keep_end);
      char* dst = kdst + row * ROW_BYTES + col * 16;
      cp_async16(dst, ksrc + (valid ? c * 8 : 0), valid);
      cp_async16(dst + TILE * ROW_BYTES, vsrc + (valid ? c * 8 : 0), valid);
    }
  }
}

// ---- the same two steps over tiles that TMA wrote: 64-column slices of [rows, 128 bytes], 128-byte swizzled
// (slice s of a tile of ROWS keys starts at s * ROWS * 128 bytes; the tile's base is 1024-byte aligned).
template <int ROWS>
__device__ __forceinline__ void qk_16keys_swizzled(const uint32_t (&q)[KSTEPS][4], const char* ktile, int row0, int lane,
                                                   float (&s)[2][4]) {
#pragma unroll
  for (int i = 0; i < 2; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
  const int mi = lane >> 3, r = lane & 7;
  const int row = row0 + (mi >> 1) * 8 + r;
#pragma unroll
  for (int ks = 0; ks < KSTEPS; ++ks) {
    uint32_t b[4];
    ldmatrix_x4(b, ktile + (ks >> 2) * ROWS * 128 + swizzled_offset(row, (ks & 3) * 2 + (mi & 1)));
    mma_bf16(s[0], q[ks], b[0], b[1]);
    mma_bf16(s[1], q[ks], b[2], b[3]);
  }
}

template <int ROWS>
__device__ __forceinline__ void softmax_pv_16keys_swizzled(WarpSoftmax& st, float (&s)[2][4], const char* vtile, int row0,
                                                           int lane) {
  float mx[2];
  mx[0] = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1]));
  mx[1] = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
  }
  float corr[2], mnew[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    mnew[h] = fmaxf(st.m[h], mx[h]);
    corr[h] = (st.m[h] == -INFINITY) ? 0.f : fast_exp2(st.m[h] - mnew[h]);
    st.m[h] = mnew[h];
  }
  float p[2][4];
  const float m0 = mnew[0] == -INFINITY ? 0.f : mnew[0], m1 = mnew[1] == -INFINITY ? 0.f : mnew[1];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    p[i][0] = fast_exp2(s[i][0] - m0);
    p[i][1] = fast_exp2(s[i][1] - m0);
    p[i][2] = fast_exp2(s[i][2] - m1);
    p[i][3] = fast_exp2(s[i][3] - m1);
  }
  st.l[0] = st.l[0] * corr[0] + (p[0][0] + p[0][1] + p[1][0] + p[1][1]);
  st.l[1] = st.l[1] * corr[1] + (p[0][2] + p[0][3] + p[1][2] + p[1][3]);
  uint32_t a[4];
  a[0] = pack_bf16(p[0][0], p[0][1]);
  a[1] = pack_bf16(p[0][2], p[0][3]);
  a[2] = pack_bf16(p[1][0], p[1][1]);
  a[3] = pack_bf16(p[1][2], p[1][3]);
  const int mi = lane >> 3, r = lane & 7;
  const int row = row0 + (mi & 1) * 8 + r;
#pragma unroll
  for (int j = 0; j < DTILES; j += 2) {
    st.o[j][0] *= corr[0]; st.o[j][1] *= corr[0]; st.o[j][2] *= corr[1]; st.o[j][3] *= corr[1];
    st.o[j + 1][0] *= corr[0]; st.o[j + 1][1] *= corr[0]; st.o[j + 1][2] *= corr[1]; st.o[j + 1][3] *= corr[1];
    const int d0 = j * 8 + (mi >> 1) * 8;      // first of the eight value columns this lane's row address names
    uint32_t b[4];
    ldmatrix_x4_trans(b, vtile + (d0 >> 6) * ROWS * 128 + swizzled_offset(row, (d0 & 63) >> 3));
    mma_bf16(st.o[j], a, b[0], b[1]);
    mma_bf16(st.o[j + 1], a, b[2], b[3]);
  }
}

// Page ids for a TMA producer warp.  A look-up is a global load with a long latency, and a producer that needs
// one per tile cannot run ahead of it; so the warp's 32 lanes fetch the pages of 32 runs of 16 keys (8 tiles) at
// once, one chunk ahead of their use, and hand them to the issuing lane by shuffle.
struct WarpPages {
  int cur = PAGE_NONE, next = PAGE_NONE;   // this lane's run in the current and in the next chunk
  // `first_key` and the runs behind it are virtual keys of `km` (positions themselves with the default map); a run is
  // wanted if it reaches into [begin, end) or lies below `keep_end`
  __device__ __forceinline__ int fetch(const int* __restrict__ table, int block_size, int first_key, int chunk, int lane,
                                       int begin, int end, KeptKeys km, int keep_end) const {
    const int key0 = km.real(first_key + (chunk * 32 + lane) * RUN_KEYS);
    return ((key0 < end && key0 + RUN_KEYS > begin) || key0 < keep_end) ? table[key0 / block_size] : PAGE_NONE;
  }
  // call with all lanes at tile `it` (tiles of 64 keys = 4 runs) before `page()`
  __device__ __forceinline__ void advance(const int* __restrict__ table, int block_size, int first_key, int it, int lane,
                                          int begin, int end, KeptKeys km = KeptKeys{0, 0}, int keep_end = 0) {
    if ((it & 7) == 0) {
      const int chunk = it >> 3;
      cur = it == 0 ? fetch(table, block_size, first_key, 0, lane, begin, end, km, keep_end) : next;
      next = fetch(table, block_size, first_key, chunk + 1, lane, begin, end, km, keep_end);
    }
  }
  // page of run `run` (0..3) of tile `it`, the same value in every lane
  __device__ __forceinline__ int page(int it, int run) const { return __shfl_sync(0xffffffffu, cur, ((it & 7) << 2) + run); }
};

}  // namespace vob
