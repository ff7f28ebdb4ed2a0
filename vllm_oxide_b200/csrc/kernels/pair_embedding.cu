// The embedding of a token plus the embedding of the pair (token before, token), hashed into buckets:
//
//     x[t] = table[id_t] + pairs[(id_{t-1} * mul_prev + id_t * mul_cur) mod buckets]        (float, one rounding at most)
//
// A sequence's first token (position 0) reads row `buckets` of the pair table, its last one.  The token before a portion's first
// comes from the request's state slot (one integer), where the portion's last token is left.  The block of a portion's first
// token does both, so that no block can overwrite what another still has to read.
#include "common.cuh"

namespace vob {

template <typename T>
__global__ void __launch_bounds__(256)
pair_embedding_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int* __restrict__ ids,
                      const int* __restrict__ positions, const int* __restrict__ token_req, const int* __restrict__ cu_q,
                      const int* __restrict__ state_slots, int* state, long state_stride, float* x, int D, int vocab, long buckets,
                      long mul_prev, long mul_cur, long num_slots, int* err) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int req = token_req[t];
  int id = ids[t];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) atomicOr(err, VOB_ERR_TOKEN_ID);
    id = 0;
  }
  long row = -1;                 // padding takes no pair
  __shared__ long shared_row;
  if (threadIdx.x == 0) {
    if (req >= 0 && pairs) {
      const int first = cu_q[req], last = cu_q[req + 1] - 1;
      int before = 0;
      if (t > first) {
        before = ids[t - 1];
      } else {
        const int slot = state_slots[req];
        if (slot < 0 || slot >= num_slots) {
          atomicOr(err, VOB_ERR_SLOT);
        } else {
          before = state[(size_t)slot * state_stride];
          state[(size_t)slot * state_stride] = ids[last];
        }
      }
      row = positions[t] == 0 ? buckets : ((long)before * mul_prev + (long)id * mul_cur) % buckets;
      if (row < 0) row += buckets;
    }
    shared_row = row;
  }
  __syncthreads();
  row = shared_row;
  const T* e = table + (size_t)id * D;
  const T* p = row >= 0 ? pairs + (size_t)row * D : nullptr;
  float* o = x + (size_t)t * D;
  for (int d = threadIdx.x; d < D; d += 256) o[d] = to_f<T>(e[d]) + (p ? to_f<T>(p[d]) : 0.f);
}

}  // namespace vob

using namespace vob;

// table [vocab, D], pairs [buckets + 1, D] of `dtype` (pairs null: the token's embedding alone); ids, positions, token_req [T];
// state int [num_slots, state_stride]; x [T, D] float.
VOB_API int vob_pair_embedding(const void* table, const void* pairs, const int* ids, const int* positions, const int* token_req,
                               const int* cu_q, const int* state_slots, int* state, long state_stride, float* x, int T, int D,
                               int vocab, long buckets, long mul_prev, long mul_cur, long num_slots, int dtype, int* err,
                               cudaStream_t stream) {
  if (T <= 0) return 0;
  if (D <= 0 || vocab <= 0 || (pairs && (buckets <= 0 || !state || state_stride < 1))) return VOB_BAD_ARGUMENT;
#define VOB_PE(TT)                                                                                                              \
  return launch_kernel(pair_embedding_kernel<TT>, dim3(T), 256, 0, stream, (const TT*)table, (const TT*)pairs, ids, positions,  \
                       token_req, cu_q, state_slots, state, state_stride, x, D, vocab, buckets, mul_prev, mul_cur, num_slots, err)
  if (dtype == VOB_F32) { VOB_PE(float); }
  if (dtype == VOB_BF16) { VOB_PE(__nv_bfloat16); }
#undef VOB_PE
  return VOB_BAD_ARGUMENT;
}
