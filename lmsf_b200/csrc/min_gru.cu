// A gated recurrence element by element whose gates read the current token only (minGRU): per request one float32 value per
// channel, kept across steps in a state slot.
//
//   z = sigmoid(raw_z + b_z);  u = raw_u + b_u;  candidate = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S_t = (1 - z) S_(t-1) + z candidate;   out_t = S_t * silu(raw_g)
//
// raw_z, raw_u and raw_g are columns of one projection's output.  The step S -> a S + b composes, (a, b) after (a', b') being
// (a a', a b' + b), so the tokens of a portion need not be walked one after the other:
//   * single tokens and short portions: a thread owns V channels of a request and walks its tokens;
//   * long portions: a block owns 32 channels of a request; 64 lanes of four consecutive tokens each compute their (a, b),
//     compose them, scan the compositions over the lanes (shuffles inside a warp, shared memory between warps) and then apply
//     them from the true state: 256 tokens a turn, one read of every input.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_min_gru)

namespace lmsf {

struct GruArgs {
  const void* z; const void* u; const void* g; long long stride;     // [n_tokens, width] each, one row stride
  const float* bz; const float* bu;                                  // [width] or null
  void* out; long long out_stride;
  float* state;                                                      // [slots, width]
  const int* cu_q; const int* state_slot;
  int width;
};

__device__ __forceinline__ float gru_sigmoid(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
// the step's (a, b) from the two logits; 1 - z is computed as sigmoid(-logit)
__device__ __forceinline__ void gru_step(float rz, float ru, float& a, float& b) {
  const float z = gru_sigmoid(rz);
  a = gru_sigmoid(-rz);
  b = z * (ru >= 0.f ? ru + 0.5f : gru_sigmoid(ru));
}

template <typename T, int V> __device__ __forceinline__ void gru_load(const T* p, float (&v)[V]) {
  if constexpr (V == 4) ld4(p, v);
  else v[0] = to_f32(*p);
}
template <typename T, int V> __device__ __forceinline__ void gru_store(T* p, const float (&v)[V]) {
  if constexpr (V == 4) st4(p, v);
  else *p = from_f32<T>(v[0]);
}

template <typename T, int V>
__global__ void __launch_bounds__(128) min_gru_walk_kernel(GruArgs a) {
  pdl_launch_dependents();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  const int seq = blockIdx.y;
  float bz[V], bu[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    bz[e] = (a.bz && c + e < a.width) ? a.bz[c + e] : 0.f;
    bu[e] = (a.bu && c + e < a.width) ? a.bu[c + e] : 0.f;
  }
  pdl_wait();
  const int t0 = a.cu_q[seq], t1 = a.cu_q[seq + 1];
  if (c >= a.width || t1 <= t0) return;
  float* slot = a.state + (size_t)a.state_slot[seq] * a.width + c;
  float S[V];
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = slot[e];
  for (int t = t0; t < t1; ++t) {
    const size_t at = (size_t)t * a.stride + c;
    float z[V], u[V], g[V], o[V];
    gru_load<T, V>((const T*)a.z + at, z);
    gru_load<T, V>((const T*)a.u + at, u);
    gru_load<T, V>((const T*)a.g + at, g);
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float m, b;
      gru_step(z[e] + bz[e], u[e] + bu[e], m, b);
      S[e] = fmaf(m, S[e], b);
      o[e] = S[e] * (g[e] * gru_sigmoid(g[e]));
    }
    gru_store<T, V>((T*)a.out + (size_t)t * a.out_stride + c, o);
  }
#pragma unroll
  for (int e = 0; e < V; ++e) slot[e] = S[e];
}

constexpr int kGruThreads = 512, kGruWarps = kGruThreads / 32;
constexpr int kGruGroups = 8;                       // groups of 4 channels per block
constexpr int kGruChannels = kGruGroups * 4;
constexpr int kGruTokens = 4;                       // consecutive tokens of a lane
constexpr int kGruTile = kGruThreads / kGruGroups * kGruTokens;     // 256

template <typename T, bool WIDE>
__global__ void __launch_bounds__(kGruThreads) min_gru_scan_kernel(GruArgs a) {
  __shared__ float wa[2][kGruWarps][kGruChannels], wb[2][kGruWarps][kGruChannels];
  __shared__ float carry[2][kGruChannels];
  const int tid = threadIdx.x, grp = tid % kGruGroups, tl = tid / kGruGroups, warp = tid >> 5, lane = tid & 31;
  const int c = blockIdx.x * kGruChannels + grp * 4, seq = blockIdx.y;
  const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
  if (n <= 0) return;
  float* slot = a.state + (size_t)a.state_slot[seq] * a.width;
  float bz[4], bu[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    bz[e] = (a.bz && c + e < a.width) ? a.bz[c + e] : 0.f;
    bu[e] = (a.bu && c + e < a.width) ? a.bu[c + e] : 0.f;
  }
  if (tid < kGruChannels) carry[0][tid] = blockIdx.x * kGruChannels + tid < a.width ? slot[blockIdx.x * kGruChannels + tid] : 0.f;
  auto load = [&](const void* base, int t, float (&v)[4]) {
    const T* p = (const T*)base + (size_t)(t0 + t) * a.stride + c;
    if (WIDE) { if (c < a.width) { ld4(p, v); return; } }
    else {
#pragma unroll
      for (int e = 0; e < 4; ++e) v[e] = c + e < a.width ? to_f32(p[e]) : 0.f;
      return;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = 0.f;
  };
  for (int base = 0, turn = 0; base < n; base += kGruTile, turn ^= 1) {
    const int t = base + tl * kGruTokens;
    float A[kGruTokens][4], B[kGruTokens][4], G[kGruTokens][4];
    float ca[4] = {1.f, 1.f, 1.f, 1.f}, cb[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < kGruTokens; ++j) {
      if (t + j < n) { load(a.z, t + j, A[j]); load(a.u, t + j, B[j]); load(a.g, t + j, G[j]); }
    }
#pragma unroll
    for (int j = 0; j < kGruTokens; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (t + j < n) {
          float m, b;
          gru_step(A[j][e] + bz[e], B[j][e] + bu[e], m, b);
          A[j][e] = m;
          B[j][e] = b;
        } else {                                    // behind the portion's end: nothing changes
          A[j][e] = 1.f;
          B[j][e] = 0.f;
        }
        cb[e] = fmaf(A[j][e], cb[e], B[j][e]);
        ca[e] *= A[j][e];
      }
    // compositions over the four lanes of tokens in a warp (inclusive), then the warp's whole
    float pa[4], pb[4];                             // the lanes before this one in the warp
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      float xa = ca[e], xb = cb[e];
#pragma unroll
      for (int off = kGruGroups; off < 32; off <<= 1) {
        const float qa = __shfl_up_sync(0xffffffffu, xa, off), qb = __shfl_up_sync(0xffffffffu, xb, off);
        if (lane >= off) { xb = fmaf(xa, qb, xb); xa *= qa; }
      }
      const float ua = __shfl_up_sync(0xffffffffu, xa, kGruGroups), ub = __shfl_up_sync(0xffffffffu, xb, kGruGroups);
      pa[e] = lane >= kGruGroups ? ua : 1.f;
      pb[e] = lane >= kGruGroups ? ub : 0.f;
      if (lane >= 32 - kGruGroups) { wa[turn][warp][grp * 4 + e] = xa; wb[turn][warp][grp * 4 + e] = xb; }
    }
    __syncthreads();
    float S[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      S[e] = carry[turn][grp * 4 + e];
      for (int w = 0; w < warp; ++w) S[e] = fmaf(wa[turn][w][grp * 4 + e], S[e], wb[turn][w][grp * 4 + e]);
      S[e] = fmaf(pa[e], S[e], pb[e]);
    }
#pragma unroll
    for (int j = 0; j < kGruTokens; ++j) {
      float o[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        S[e] = fmaf(A[j][e], S[e], B[j][e]);
        o[e] = t + j < n ? S[e] * (G[j][e] * gru_sigmoid(G[j][e])) : 0.f;
      }
      if (t + j < n) {
        T* p = (T*)a.out + (size_t)(t0 + t + j) * a.out_stride + c;
        if (WIDE) { if (c < a.width) st4(p, o); }
        else {
#pragma unroll
          for (int e = 0; e < 4; ++e) if (c + e < a.width) p[e] = from_f32<T>(o[e]);
        }
      }
    }
    // the last lane of tokens holds the state after the turn; the next turn writes the other halves of the shared arrays,
    // and the barrier in it stands between these writes and their readers
    if (tl == kGruThreads / kGruGroups - 1) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        carry[turn ^ 1][grp * 4 + e] = S[e];
        if (base + kGruTile >= n && c + e < a.width) slot[c + e] = S[e];
      }
    }
  }
}

}  // namespace lmsf

// z, u, g: [n_tokens, width] of `dtype`, one row stride; out likewise with its own; bz, bu: float32 [width] or null; state:
// float32 [slots, width].  max_q: the longest portion of the launch (the host's copy; chooses the kernel).
LMSF_API int lmsf_min_gru(const void* z, const void* u, const void* g, long long stride, const float* bz, const float* bu,
                          void* out, long long out_stride, float* state, const int* cu_q, const int* state_slot, int n_seqs,
                          int max_q, int width, int dtype, void* stream) {
  using namespace lmsf;
  if (n_seqs <= 0 || max_q <= 0) return 0;
  if (width <= 0 || stride < width || out_stride < width) LMSF_REFUSE("min_gru: width=%d, row strides %lld and %lld", width, stride, out_stride);
  if (n_seqs > 65535) LMSF_REFUSE("min_gru: more than 65535 requests in one launch");
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("min_gru: unknown dtype code %d", dtype);
  GruArgs a{z, u, g, stride, bz, bu, out, out_stride, state, cu_q, state_slot, width};
  cudaStream_t s = (cudaStream_t)stream;
  const size_t el = dtype == LMSF_F32 ? 4 : 2;
  const bool wide = width % 4 == 0 && stride % 4 == 0 && out_stride % 4 == 0 &&
                    ((uintptr_t)z | (uintptr_t)u | (uintptr_t)g | (uintptr_t)out) % (4 * el) == 0;
  if (max_q <= 16) {
    const dim3 grid(ceil_div(width, 128 * (wide ? 4 : 1)), n_seqs);
    if (dtype == LMSF_F32) return wide ? launch_pdl(min_gru_walk_kernel<float, 4>, grid, dim3(128), 0, s, a)
                                       : launch_pdl(min_gru_walk_kernel<float, 1>, grid, dim3(128), 0, s, a);
    return wide ? launch_pdl(min_gru_walk_kernel<bf16, 4>, grid, dim3(128), 0, s, a)
                : launch_pdl(min_gru_walk_kernel<bf16, 1>, grid, dim3(128), 0, s, a);
  }
  const dim3 grid(ceil_div(width, kGruChannels), n_seqs);
  if (dtype == LMSF_F32) {
    if (wide) min_gru_scan_kernel<float, true><<<grid, kGruThreads, 0, s>>>(a);
    else min_gru_scan_kernel<float, false><<<grid, kGruThreads, 0, s>>>(a);
  } else {
    if (wide) min_gru_scan_kernel<bf16, true><<<grid, kGruThreads, 0, s>>>(a);
    else min_gru_scan_kernel<bf16, false><<<grid, kGruThreads, 0, s>>>(a);
  }
  return LMSF_LAUNCH_STATUS();
}
