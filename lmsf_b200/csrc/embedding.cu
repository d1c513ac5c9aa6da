// Embedding gather: out[t, :] = table[ids[t], :].
// Counterpart in the reference: index_select in
// core/src/model_executor/layers/vocab_parallel_embedding.rs:28-37.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_embedding)

namespace lmsf {

// One block per token.  Rows are copied as 16-byte words when the row size allows it.
// An id outside [0, vocab) writes a row of zeros and raises *error_flag (never reads outside the table).
template <typename W>
__global__ void embedding_kernel(W* __restrict__ out, const W* __restrict__ table, const int* __restrict__ ids,
                                 int row_words, int vocab, int* __restrict__ error_flag) {
  const int t = blockIdx.x;
  const int id = ids[t];
  W* dst = out + (size_t)t * row_words;
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0 && error_flag) atomicExch(error_flag, 1);
    W zero;
    memset(&zero, 0, sizeof(W));
    for (int i = threadIdx.x; i < row_words; i += blockDim.x) dst[i] = zero;
    return;
  }
  const W* src = table + (size_t)id * row_words;
  for (int i = threadIdx.x; i < row_words; i += blockDim.x) dst[i] = src[i];
}

// The same with every value multiplied by `scale` (float32 product, rounded once): the embedding scale that some
// architectures apply to their input (sqrt of the width, for one).
template <typename T>
__global__ void embedding_scaled_kernel(T* __restrict__ out, const T* __restrict__ table, const int* __restrict__ ids,
                                        int hidden, int vocab, float scale, int* __restrict__ error_flag) {
  const int t = blockIdx.x;
  const int id = ids[t];
  T* dst = out + (size_t)t * hidden;
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0 && error_flag) atomicExch(error_flag, 1);
  const T* src = table + (size_t)(ok ? id : 0) * hidden;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = ok ? from_f32<T>(to_f32(src[i]) * scale) : from_f32<T>(0.f);
}

// The same as the start of a float32 residual stream: the product is not rounded, whatever the table's type.
template <typename T, int V>
__global__ void embedding_stream_kernel(float* __restrict__ out, const T* __restrict__ table, const int* __restrict__ ids,
                                        int hidden, int vocab, float scale, int* __restrict__ error_flag) {
  const int t = blockIdx.x;
  const int id = ids[t];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0 && error_flag) atomicExch(error_flag, 1);
  const T* src = table + (size_t)(ok ? id : 0) * hidden;
  float* dst = out + (size_t)t * hidden;
  for (int i = threadIdx.x * V; i < hidden; i += blockDim.x * V) {
    if constexpr (V == 4) {
      float x[4];
      ld4(src + i, x);
#pragma unroll
      for (int k = 0; k < 4; ++k) x[k] = ok ? x[k] * scale : 0.f;
      st4(dst + i, x);
    } else {
      dst[i] = ok ? to_f32(src[i]) * scale : 0.f;
    }
  }
}

// out[t, :] = table[id_t, :] * scale + pairs[row_t, :] in float32, where row_t = (id_{t-1} * mul_prev + id_t * mul_cur) mod buckets
// is chosen by the token and the token before it in the same request, and row `buckets` (the table's last) belongs to a
// request's first token.  The token before a portion's first token is the request's state: last[slot], one int32 per state
// slot.  The block of a portion's first token reads it and then stores the portion's last token there; no other block touches
// that slot, so the launch needs no second pass.  One block per token.
template <typename T, bool VEC>
__global__ void embedding_pairs_kernel(float* __restrict__ out, const T* __restrict__ table, const T* __restrict__ pairs,
                                       const int* __restrict__ ids, const int* __restrict__ positions,
                                       const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                                       const int* __restrict__ state_slot, int* __restrict__ last, int hidden, int vocab,
                                       int buckets, long long mul_prev, long long mul_cur, float scale,
                                       int* __restrict__ error_flag) {
  __shared__ int s_prev;
  const int t = blockIdx.x;
  const int id = ids[t];
  const int seq = token_seq[t];
  const bool starts = t == cu_q[seq];
  if (threadIdx.x == 0) {
    int prev;
    if (starts) {
      const int slot = state_slot[seq];
      prev = last[slot];
      last[slot] = ids[cu_q[seq + 1] - 1];
    } else {
      prev = ids[t - 1];
    }
    s_prev = positions[t] == 0 ? -1 : prev;
  }
  __syncthreads();
  const int prev = s_prev;
  const bool ok = id >= 0 && id < vocab && prev < vocab;
  if (!ok && threadIdx.x == 0 && error_flag) atomicExch(error_flag, 1);
  const long long row = prev < 0 ? buckets : ((long long)prev * mul_prev + (long long)id * mul_cur) % buckets;
  const T* src = table + (size_t)(ok ? id : 0) * hidden;
  const T* pr = pairs + (size_t)(ok ? row : buckets) * hidden;
  float* dst = out + (size_t)t * hidden;
  if constexpr (VEC) {   // four values an access: widths that 4 divides, aligned tables
    for (int i = threadIdx.x * 4; i < hidden; i += blockDim.x * 4) {
      float a[4], b[4], r[4];
      ld4(src + i, a);
      ld4(pr + i, b);
#pragma unroll
      for (int k = 0; k < 4; ++k) r[k] = ok ? fmaf(a[k], scale, b[k]) : 0.f;
      st4(dst + i, r);
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) dst[i] = ok ? fmaf(to_f32(src[i]), scale, to_f32(pr[i])) : 0.f;
  }
}

// token_ids[dst[i]] = source[src[i]] for every i with dst[i] >= 0: puts tokens that were sampled on the device
// into the next step's input without a round trip to the host.
__global__ void patch_tokens_kernel(int* __restrict__ token_ids, const int* __restrict__ dst, const int* __restrict__ src,
                                    const int* __restrict__ source, int n) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n && dst[i] >= 0) token_ids[dst[i]] = source[src[i]];
}

}  // namespace lmsf

LMSF_API int lmsf_patch_tokens(int* token_ids, const int* dst, const int* src, const int* source, int n, void* stream) {
  if (n <= 0) return 0;
  lmsf::patch_tokens_kernel<<<(n + 127) / 128, 128, 0, (cudaStream_t)stream>>>(token_ids, dst, src, source, n);
  return LMSF_LAUNCH_STATUS();
}

LMSF_API int lmsf_embedding(void* out, const void* table, const int* ids, int n_tokens, int hidden, int vocab,
                            int dtype, int* error_flag, void* stream) {
  using namespace lmsf;
  if (n_tokens <= 0) return 0;
  if (hidden <= 0 || vocab <= 0) LMSF_REFUSE("embedding: hidden=%d vocab=%d must be positive", hidden, vocab);
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("embedding: unknown dtype code %d", dtype);
  const size_t row_bytes = (size_t)hidden * (dtype == LMSF_F32 ? 4 : 2);
  cudaStream_t s = (cudaStream_t)stream;
  const bool aligned16 = row_bytes % 16 == 0 && ((uintptr_t)out % 16 == 0) && ((uintptr_t)table % 16 == 0);
  if (aligned16) {
    const int words = (int)(row_bytes / 16);
    const int threads = words >= 256 ? 256 : (words >= 64 ? 64 : 32);
    embedding_kernel<uint4><<<n_tokens, threads, 0, s>>>((uint4*)out, (const uint4*)table, ids, words, vocab,
                                                          error_flag);
  } else if (dtype == LMSF_F32) {
    embedding_kernel<float><<<n_tokens, 128, 0, s>>>((float*)out, (const float*)table, ids, hidden, vocab, error_flag);
  } else {
    embedding_kernel<unsigned short><<<n_tokens, 128, 0, s>>>((unsigned short*)out, (const unsigned short*)table, ids,
                                                               hidden, vocab, error_flag);
  }
  return LMSF_LAUNCH_STATUS();
}

LMSF_API int lmsf_embedding_scaled(void* out, const void* table, const int* ids, int n_tokens, int hidden, int vocab,
                                   float scale, int dtype, int* error_flag, void* stream) {
  using namespace lmsf;
  if (n_tokens <= 0) return 0;
  if (hidden <= 0 || vocab <= 0) LMSF_REFUSE("embedding: hidden=%d vocab=%d must be positive", hidden, vocab);
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("embedding: unknown dtype code %d", dtype);
  cudaStream_t s = (cudaStream_t)stream;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (dtype == LMSF_F32)
    embedding_scaled_kernel<float><<<n_tokens, threads, 0, s>>>((float*)out, (const float*)table, ids, hidden, vocab, scale, error_flag);
  else
    embedding_scaled_kernel<bf16><<<n_tokens, threads, 0, s>>>((bf16*)out, (const bf16*)table, ids, hidden, vocab, scale, error_flag);
  return LMSF_LAUNCH_STATUS();
}

// out: float32 [n_tokens, hidden]; table: [vocab, hidden] and pairs: [buckets + 1, hidden] of `dtype`; last: int32, one per
// state slot (the slot's newest token).  mul_prev, mul_cur >= 0.
LMSF_API int lmsf_embedding_pairs(float* out, const void* table, const void* pairs, const int* ids, const int* positions,
                                  const int* token_seq, const int* cu_q, const int* state_slot, int* last, int n_tokens,
                                  int hidden, int vocab, int buckets, long long mul_prev, long long mul_cur, float scale,
                                  int dtype, int* error_flag, void* stream) {
  using namespace lmsf;
  if (n_tokens <= 0) return 0;
  if (hidden <= 0 || vocab <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0)
    LMSF_REFUSE("embedding: hidden=%d vocab=%d buckets=%d and non-negative multipliers", hidden, vocab, buckets);
  if ((double)vocab * (double)mul_prev + (double)vocab * (double)mul_cur > 9.0e18)
    LMSF_REFUSE("embedding: the pair index overflows 64 bits");
  cudaStream_t s = (cudaStream_t)stream;
  const int threads = hidden >= 1024 ? 256 : 128;
  const size_t esize = dtype == LMSF_F32 ? 4 : 2;
  const bool vec = hidden % 4 == 0 && (uintptr_t)out % 16 == 0 && ((uintptr_t)table | (uintptr_t)pairs) % (4 * esize) == 0;
#define LMSF_EP(T, V) embedding_pairs_kernel<T, V><<<n_tokens, threads, 0, s>>>(out, (const T*)table, (const T*)pairs, ids, positions, \
    token_seq, cu_q, state_slot, last, hidden, vocab, buckets, mul_prev, mul_cur, scale, error_flag)
  if (dtype == LMSF_F32) { if (vec) LMSF_EP(float, true); else LMSF_EP(float, false); }
  else if (dtype == LMSF_BF16) { if (vec) LMSF_EP(bf16, true); else LMSF_EP(bf16, false); }
  else LMSF_REFUSE("embedding: unknown dtype code %d", dtype);
#undef LMSF_EP
  return LMSF_LAUNCH_STATUS();
}

// out: float32 [n, hidden] = table[ids] * scale, the start of a float32 residual stream; table: [vocab, hidden] of `dtype`.
LMSF_API int lmsf_embedding_stream(float* out, const void* table, const int* ids, int n, int hidden, int vocab, float scale,
                                   int dtype, int* error_flag, void* stream) {
  using namespace lmsf;
  if (n <= 0) return 0;
  if (hidden <= 0 || vocab <= 0) LMSF_REFUSE("embedding_stream: hidden=%d vocab=%d", hidden, vocab);
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("embedding_stream: unknown dtype code %d", dtype);
  cudaStream_t s = (cudaStream_t)stream;
  const int threads = hidden >= 1024 ? 256 : 64;
  const bool wide = hidden % 4 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)table % (dtype == LMSF_F32 ? 16 : 8) == 0;
#define LMSF_GO(T, V) embedding_stream_kernel<T, V><<<n, threads, 0, s>>>(out, (const T*)table, ids, hidden, vocab, scale, error_flag)
  if (dtype == LMSF_F32) { if (wide) LMSF_GO(float, 4); else LMSF_GO(float, 1); }
  else { if (wide) LMSF_GO(bf16, 4); else LMSF_GO(bf16, 1); }
#undef LMSF_GO
  return LMSF_LAUNCH_STATUS();
}
