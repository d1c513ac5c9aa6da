// Causal attention of any mix of prompt portions and decoded tokens over the paged cache:
// the plain twin of the fast kernels, and the kernel of the float32 path.
//
// Counterparts in the reference: the dense prompt attention of
// core/src/model_executor/layers/attention.rs:106-159 and paged_attention_v1_kernel,
// vllm/kernels/attention/attention_kernels.cu:82-414.  Differences: one kernel serves prompt
// portions and decoded tokens alike (every query token reads its keys from pages, its own key
// included, which the cache write has stored before); the softmax is exact (no 1e-6 in the
// denominator, expf rather than __expf); any head size that is a multiple of 16 up to 640.
//
// One block of 4 warps per (query token, query head).  Keys are walked in tiles of 32 that are
// aligned to absolute positions; tile j belongs to warp j % 4; every warp keeps a running
// (max, sum, accumulator) and the four are merged in a fixed order.  The order of every
// floating-point operation therefore depends on the token's position only, not on how the
// tokens were cut into steps, which requests share the batch or which pages hold the keys.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_attention_generic)

namespace lmsf {

constexpr int kMaxHeadDim = 640;
constexpr int kWarps = 4;

struct GenericAttnArgs {
  const void* q; long long q_stride;           // [n_tokens, n_q_heads, hd]
  void* out; long long out_stride;             // [n_tokens, n_q_heads, hd]
  const void* cache; long long page_stride;    // [page][2][kv_head][slot][hd]
  const int* block_table; int max_blocks; int block_size;
  const int* token_seq; const int* positions;
  float scale; int window;                     // window <= 0: all keys
  int n_q_heads, n_kv_heads, head_dim;
  float softcap;                               // > 0: scores become softcap * tanh(score / softcap) before the softmax
  const float* slopes;                         // [n_q_heads] or null: slope * (key position - query position) is added to the scores
  int shared_kv;                               // 1: a page holds one vector per token that is key and value at once ([page][1][kv_head][slot][hd])
  const void* gate; long long gate_stride;     // [n_tokens, n_q_heads] or null: head h's output is multiplied by sigmoid(gate[t, h])
  int chunk;                                   // > 0: a query at position p sees the keys from p - p % chunk on (its own chunk of positions)
  const float* log_r1; const float* log_r2;    // [n_q_heads] or null: r1 * log(1 + r2 * (query position - key position)) is taken off the scores
  const float* sinks;                          // [n_q_heads] or null: exp(sink) joins the softmax's denominator, without a key or a value
  int keep_first;                              // > 0 (with a window): the first keep_first keys of the request stay visible behind the window
  int sigmoid;                                 // 1: a key's weight is sigmoid(score), not normalised over the keys (no softmax)
  const float* head_bias;                      // [n_q_heads] or null: a number per query head added to every scaled score
  const float* dist; int dist_n;               // [n_q_heads][dist_n] or null: the entry of (query position - key position), the last for larger ones, is added
};

// MAXD: the largest head size of a build (accumulators in registers)
template <typename T, int MAXD>
__global__ void __launch_bounds__(kWarps * 32) attention_generic_kernel(GenericAttnArgs a) {
  __shared__ float qs[MAXD];
  __shared__ float part_acc[kWarps][MAXD];
  __shared__ float part_m[kWarps], part_l[kWarps];

  const int t = blockIdx.x, head = blockIdx.y;
  const int hd = a.head_dim;
  const int kvh = head / (a.n_q_heads / a.n_kv_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int pos = a.positions[t];
  int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  if (a.chunk > 0) lo = max(lo, pos - pos % a.chunk);
  const int keep = lo > 0 ? min(a.keep_first, lo) : 0;   // keys 0 .. keep - 1 are seen although the window has passed them
  const float hb = a.head_bias ? a.head_bias[head] : 0.f;
  const int* table = a.block_table + (size_t)a.token_seq[t] * a.max_blocks;

  const T* q = (const T*)a.q + (size_t)t * a.q_stride + (size_t)head * hd;
  for (int d = threadIdx.x; d < hd; d += blockDim.x) qs[d] = to_f32(q[d]);
  __syncthreads();

  const size_t head_off = (size_t)kvh * a.block_size * hd;
  const size_t v_off = a.shared_kv ? 0 : (size_t)a.n_kv_heads * a.block_size * hd;
  const int nd = (hd + 31) / 32;

  float m = -INFINITY, l = 0.f;
  float acc[MAXD / 32];
#pragma unroll
  for (int i = 0; i < MAXD / 32; ++i) acc[i] = 0.f;

  // tiles 0 .. (keep - 1) / 32 hold the kept first keys, tiles lo / 32 .. pos / 32 the window; tile j is always warp j % 4's
  const int first_tile = keep > 0 ? 0 : lo / 32;
  for (int tile = first_tile + ((warp - first_tile) % kWarps + kWarps) % kWarps; tile * 32 <= pos; tile += kWarps) {
    if (tile * 32 >= keep && tile < lo / 32) {   // between the kept keys and the window: on to this warp's first tile of the window
      tile += (lo / 32 - tile - 1) / kWarps * kWarps;
      continue;
    }
    const int key = tile * 32 + lane;
    const bool valid = (key >= lo || key < keep) && key <= pos;
    long long row = -1;  // element offset of this lane's key row inside the layer's cache
    float s = -INFINITY;
    if (valid) {
      const int page = table[key / a.block_size];
      if (page >= 0) {  // a key without a page (a fault of the caller) is left out, never read
        row = (long long)page * a.page_stride + head_off + (size_t)(key % a.block_size) * hd;
        const T* kr = (const T*)a.cache + row;
        float dot = 0.f;
        for (int d = 0; d < hd; ++d) dot = fmaf(qs[d], to_f32(kr[d]), dot);
        s = dot * a.scale;
        if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
        if (a.slopes) s = fmaf(a.slopes[head], (float)(key - pos), s);
        if (a.log_r1) s -= a.log_r1[head] * logf(1.0f + a.log_r2[head] * (float)(pos - key));
        if (a.dist) s += a.dist[(size_t)head * a.dist_n + min(pos - key, a.dist_n - 1)];
        s += hb;
      }
    }
    if (a.sigmoid) {   // every key on its own: no running maximum, no denominator
      const float p = row >= 0 ? 1.0f / (1.0f + expf(-s)) : 0.f;
      for (int j = 0; j < 32; ++j) {
        const float pj = __shfl_sync(0xffffffffu, p, j);
        const long long rj = __shfl_sync(0xffffffffu, row, j);
        if (rj < 0) continue;
        const T* vr = (const T*)a.cache + rj + v_off;
#pragma unroll
        for (int i = 0; i < MAXD / 32; ++i) {
          const int d = lane + 32 * i;
          if (i < nd && d < hd) acc[i] = fmaf(pj, to_f32(vr[d]), acc[i]);
        }
      }
      continue;
    }
    const float m_new = fmaxf(m, warp_max(s));
    if (m_new == -INFINITY) continue;  // nothing seen yet (uniform over the warp)
    const float p = row >= 0 ? expf(s - m_new) : 0.f;
    const float alpha = expf(m - m_new);  // m = -inf on the first tile gives 0
    l = l * alpha + warp_sum(p);
#pragma unroll
    for (int i = 0; i < MAXD / 32; ++i) acc[i] *= alpha;
    for (int j = 0; j < 32; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const long long rj = __shfl_sync(0xffffffffu, row, j);
      if (rj < 0) continue;  // same for the whole warp
      const T* vr = (const T*)a.cache + rj + v_off;
#pragma unroll
      for (int i = 0; i < MAXD / 32; ++i) {
        const int d = lane + 32 * i;
        if (i < nd && d < hd) acc[i] = fmaf(pj, to_f32(vr[d]), acc[i]);
      }
    }
    m = m_new;
  }

  if (lane == 0) { part_m[warp] = m; part_l[warp] = l; }
#pragma unroll
  for (int i = 0; i < MAXD / 32; ++i) {
    const int d = lane + 32 * i;
    if (i < nd && d < hd) part_acc[warp][d] = acc[i];
  }
  __syncthreads();

  float M = part_m[0];
  for (int w = 1; w < kWarps; ++w) M = fmaxf(M, part_m[w]);
  const float sink = a.sinks ? a.sinks[head] : -INFINITY;
  M = fmaxf(M, sink);
  float L = a.sinks ? expf(sink - M) : 0.f;
  float f[kWarps];
  for (int w = 0; w < kWarps; ++w) {
    f[w] = part_m[w] == -INFINITY ? 0.f : expf(part_m[w] - M);
    L = fmaf(part_l[w], f[w], L);
  }
  if (a.sigmoid) {   // the warps' sums are added as they are, in the order of the warps
    for (int w = 0; w < kWarps; ++w) f[w] = 1.f;
    L = 1.f;
  }
  T* o = (T*)a.out + (size_t)t * a.out_stride + (size_t)head * hd;
  const float g = a.gate ? 1.0f / (1.0f + expf(-to_f32(((const T*)a.gate)[(size_t)t * a.gate_stride + head]))) : 1.0f;
  for (int d = threadIdx.x; d < hd; d += blockDim.x) {
    float v = 0.f;
    for (int w = 0; w < kWarps; ++w) v = fmaf(part_acc[w][d], f[w], v);
    o[d] = from_f32<T>(a.gate ? (v / L) * g : v / L);
  }
}

}  // namespace lmsf

// Two changes to the scores that some architectures make and only this kernel takes.  softcap > 0: the scaled scores
// are capped smoothly, softcap * tanh(score / softcap).  slopes ([n_q_heads] float32, may be null): a position encoding
// by a bias that grows with distance, slope[head] * (key position - query position), added to the scaled score as the
// reference's decode kernel adds it (vllm/kernels/attention/attention_kernels.cu:144-145, :232-234).
// shared_kv = 1: the cache holds one vector per token and kv head, [page][1][kv_head][slot][head_dim], which is read as
// the key and as the value (attention over a cached low-rank vector).  gate ([n_tokens, n_q_heads] of `dtype`, row stride
// gate_stride, may be null): head h's output of token t is multiplied by sigmoid(gate[t, h]).
// chunk > 0: a query at position p sees only the keys of its own chunk of positions, p - p % chunk .. p (chunks are counted
// from position 0 of the request).  log_r1, log_r2 ([n_q_heads] float32, both or neither): r1 * log(1 + r2 * distance) is
// taken off the scaled score.  sinks ([n_q_heads] float32 or null): exp(sink[head]) is one more term of the denominator.
// keep_first > 0 (with a window): the request's first keep_first keys stay visible when the window has passed them, at their
// true positions.  sigmoid = 1: a visible key's weight is sigmoid(score) and the weights are not normalised (no softmax; sinks
// have no meaning then).  head_bias ([n_q_heads] float32 or null): added to every scaled score of its head.
// dist ([n_q_heads][dist_n] float32 or null): a table of what is added to the scaled score by (query position - key position);
// its last entry serves every larger distance.
LMSF_API int lmsf_attention_generic_dist(const void* q, long long q_stride, void* out, long long out_stride,
                                         const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                         int block_size, const int* token_seq, const int* positions, float scale,
                                         float softcap, const float* slopes, int window, int n_tokens, int n_q_heads,
                                         int n_kv_heads, int head_dim, int dtype, int shared_kv, const void* gate,
                                         long long gate_stride, int chunk, const float* log_r1, const float* log_r2,
                                         const float* sinks, int keep_first, int sigmoid, const float* head_bias,
                                         const float* dist, int dist_n, void* stream) {
  using namespace lmsf;
  if (n_tokens <= 0) return 0;
  if (head_dim <= 0 || head_dim > kMaxHeadDim || head_dim % 16)
    LMSF_REFUSE("attention: head_dim=%d must be a multiple of 16 between 16 and %d", head_dim, kMaxHeadDim);
  if (n_q_heads <= 0 || n_kv_heads <= 0 || n_q_heads % n_kv_heads)
    LMSF_REFUSE("attention: %d query heads cannot be grouped over %d kv heads", n_q_heads, n_kv_heads);
  if (n_q_heads > 65535) LMSF_REFUSE("attention: more than 65535 query heads");
  if (block_size <= 0 || max_blocks <= 0) LMSF_REFUSE("attention: bad block table geometry");
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("attention: unknown dtype code %d", dtype);
  if ((log_r1 == nullptr) != (log_r2 == nullptr)) LMSF_REFUSE("attention: the logarithmic bias needs both of its constants");
  GenericAttnArgs a{q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                    token_seq, positions, scale, window, n_q_heads, n_kv_heads, head_dim, softcap > 0.f ? softcap : 0.f, slopes,
                    shared_kv ? 1 : 0, gate, gate_stride, chunk > 0 ? chunk : 0, log_r1, log_r2, sinks,
                    (window > 0 && keep_first > 0) ? keep_first : 0, sigmoid ? 1 : 0, head_bias, dist, dist_n};
  if (dist && dist_n <= 0) LMSF_REFUSE("attention: a table of %d distances", dist_n);
  if (sigmoid && sinks) LMSF_REFUSE("attention: sinks belong to a softmax, not to sigmoid weights");
  dim3 grid(n_tokens, n_q_heads);
  cudaStream_t s = (cudaStream_t)stream;
#define LMSF_GO(D) do { if (dtype == LMSF_F32) attention_generic_kernel<float, D><<<grid, kWarps * 32, 0, s>>>(a); \
                        else attention_generic_kernel<bf16, D><<<grid, kWarps * 32, 0, s>>>(a); } while (0)
  if (head_dim <= 128) LMSF_GO(128);
  else if (head_dim <= 256) LMSF_GO(256);
  else LMSF_GO(kMaxHeadDim);
#undef LMSF_GO
  return LMSF_LAUNCH_STATUS();
}

LMSF_API int lmsf_attention_generic_weights(const void* q, long long q_stride, void* out, long long out_stride,
                                            const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                            int block_size, const int* token_seq, const int* positions, float scale,
                                            float softcap, const float* slopes, int window, int n_tokens, int n_q_heads,
                                            int n_kv_heads, int head_dim, int dtype, int shared_kv, const void* gate,
                                            long long gate_stride, int chunk, const float* log_r1, const float* log_r2,
                                            const float* sinks, int keep_first, int sigmoid, const float* head_bias,
                                            void* stream) {
  return lmsf_attention_generic_dist(q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                                     token_seq, positions, scale, softcap, slopes, window, n_tokens, n_q_heads, n_kv_heads,
                                     head_dim, dtype, shared_kv, gate, gate_stride, chunk, log_r1, log_r2, sinks, keep_first,
                                     sigmoid, head_bias, nullptr, 0, stream);
}

LMSF_API int lmsf_attention_generic_masked(const void* q, long long q_stride, void* out, long long out_stride,
                                           const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                           int block_size, const int* token_seq, const int* positions, float scale,
                                           float softcap, const float* slopes, int window, int n_tokens, int n_q_heads,
                                           int n_kv_heads, int head_dim, int dtype, int shared_kv, const void* gate,
                                           long long gate_stride, int chunk, const float* log_r1, const float* log_r2,
                                           const float* sinks, void* stream) {
  return lmsf_attention_generic_weights(q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                                        token_seq, positions, scale, softcap, slopes, window, n_tokens, n_q_heads, n_kv_heads,
                                        head_dim, dtype, shared_kv, gate, gate_stride, chunk, log_r1, log_r2, sinks, 0, 0, nullptr,
                                        stream);
}

LMSF_API int lmsf_attention_generic_ext(const void* q, long long q_stride, void* out, long long out_stride,
                                        const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                        int block_size, const int* token_seq, const int* positions, float scale,
                                        float softcap, const float* slopes, int window, int n_tokens, int n_q_heads,
                                        int n_kv_heads, int head_dim, int dtype, int shared_kv, const void* gate,
                                        long long gate_stride, void* stream) {
  return lmsf_attention_generic_masked(q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                                       token_seq, positions, scale, softcap, slopes, window, n_tokens, n_q_heads, n_kv_heads,
                                       head_dim, dtype, shared_kv, gate, gate_stride, 0, nullptr, nullptr, nullptr, stream);
}

LMSF_API int lmsf_attention_generic_scores(const void* q, long long q_stride, void* out, long long out_stride,
                                           const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                           int block_size, const int* token_seq, const int* positions, float scale,
                                           float softcap, const float* slopes, int window, int n_tokens, int n_q_heads,
                                           int n_kv_heads, int head_dim, int dtype, void* stream) {
  return lmsf_attention_generic_ext(q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                                    token_seq, positions, scale, softcap, slopes, window, n_tokens, n_q_heads, n_kv_heads,
                                    head_dim, dtype, 0, nullptr, 0, stream);
}

LMSF_API int lmsf_attention_generic(const void* q, long long q_stride, void* out, long long out_stride,
                                    const void* cache, long long page_stride, const int* block_table, int max_blocks,
                                    int block_size, const int* token_seq, const int* positions, float scale,
                                    int window, int n_tokens, int n_q_heads, int n_kv_heads, int head_dim, int dtype,
                                    void* stream) {
  return lmsf_attention_generic_scores(q, q_stride, out, out_stride, cache, page_stride, block_table, max_blocks, block_size,
                                       token_seq, positions, scale, 0.f, nullptr, window, n_tokens, n_q_heads, n_kv_heads,
                                       head_dim, dtype, stream);
}
