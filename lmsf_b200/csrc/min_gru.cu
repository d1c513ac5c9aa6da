// A gated recurrence element by element whose gates read the current token only (minGRU): per request one float32 value per
// channel, kept across steps in a state slot.
//
//   z = sigmoid(raw_z + b_z);  u = raw_u + b_u;  candidate = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S_t = (1 - z) S_(t-1) + z candidate;   out_t = S_t * silu(raw_g)
//
// raw_z, raw_u and raw_g are columns of one projection's output.  The step S -> a S + b composes, (a, b) after (a', b') being
// (a a', a b' + b), so the tokens of a portion need not be walked one after the other:
//   * single tokens and short portions: a thread owns V channels of a request and walks its tokens;
//   * long portions: a cluster of eight blocks owns 64 channels of a request and up to 2,048 tokens a turn.  A thread walks up
//     to 16 consecutive tokens of four channels twice: first from the identity, which gives the composition of its tokens;
//     the compositions are folded over the threads (shared memory) and over the blocks (distributed shared memory); then from
//     the true state, writing the outputs (the second read of the inputs comes from the caches; keeping the steps in registers
//     instead was slower, 51 us against 39 for 2,048 tokens of 4,096 channels, for want of resident warps).
#include <cooperative_groups.h>

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

// sigmoid(x) and sigmoid(-x) from e = exp(-|x|): the larger is 1 / (1 + e), the smaller e times it, so neither is a difference
// (2^x and 1/x of the special-function unit, each within two units of the last place)
__device__ __forceinline__ void gru_sigmoids(float x, float& pos, float& neg) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-1.4426950408889634f * fabsf(x)));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
  const float small = e * r;
  pos = x >= 0.f ? r : small;
  neg = x >= 0.f ? small : r;
}
__device__ __forceinline__ float gru_sigmoid(float x) {
  float p, n;
  gru_sigmoids(x, p, n);
  return p;
}
// the step's (a, b) from the two logits
__device__ __forceinline__ void gru_step(float rz, float ru, float& a, float& b) {
  float z;
  gru_sigmoids(rz, z, a);
  b = z * (ru >= 0.f ? ru + 0.5f : gru_sigmoid(ru));
}

template <typename T, int V> __device__ __forceinline__ void gru_load(const T* p, float (&v)[V]) {
  if constexpr (V == 4) {      // (the inputs are never written by these kernels: their loads may move past the stores)
    if constexpr (sizeof(T) == 2) {
      const uint2 x = __ldg(reinterpret_cast<const uint2*>(p));
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.x)), g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x.y));
      v[0] = f.x; v[1] = f.y; v[2] = g.x; v[3] = g.y;
    } else {
      const float4 x = __ldg(reinterpret_cast<const float4*>(p));
      v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
    }
  } else v[0] = to_f32(*p);
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

constexpr int kGruThreads = 256;
constexpr int kGruVec = 4;                          // channels of a thread
constexpr int kGruGroups = 16;                      // threads side by side over the channels
constexpr int kGruChannels = kGruGroups * kGruVec;  // 64
constexpr int kGruLanes = kGruThreads / kGruGroups; // threads side by side over the tokens
constexpr int kGruTokens = 16;                       // most consecutive tokens of a thread and turn
constexpr int kGruRanks = 8;                        // blocks of a cluster, in the order of their tokens

// WIDE: the rows take accesses of four channels
template <typename T, bool WIDE>
__global__ void __cluster_dims__(1, 1, kGruRanks) __launch_bounds__(kGruThreads) min_gru_scan_kernel(GruArgs a) {
  __shared__ float fa[kGruLanes][kGruChannels], fb[kGruLanes][kGruChannels];   // compositions of the lanes, then of those before
  __shared__ float tot[2][2][kGruChannels];         // the block's whole composition (a, b), by turn: read by the cluster
  __shared__ float start[kGruChannels];             // the state before the block's tokens
  namespace cg = cooperative_groups;
  cg::cluster_group cluster = cg::this_cluster();
  const int tid = threadIdx.x, grp = tid % kGruGroups, tl = tid / kGruGroups, rank = blockIdx.z;
  const int c = blockIdx.x * kGruChannels + grp * kGruVec, seq = blockIdx.y;
  const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
  if (n <= 0) return;                               // the same for every block of the cluster
  float* slot = a.state + (size_t)a.state_slot[seq] * a.width;
  float bz[kGruVec], bu[kGruVec];
#pragma unroll
  for (int e = 0; e < kGruVec; ++e) {
    bz[e] = (a.bz && c + e < a.width) ? a.bz[c + e] : 0.f;
    bu[e] = (a.bu && c + e < a.width) ? a.bu[c + e] : 0.f;
  }
  const int my_channel = blockIdx.x * kGruChannels + tid;
  float carry = (tid < kGruChannels && my_channel < a.width) ? slot[my_channel] : 0.f;      // one channel a thread
  const bool live = c < a.width;
  auto load = [&](const void* base, int t, float (&v)[kGruVec]) {
    const T* p = (const T*)base + (size_t)(t0 + t) * a.stride + c;
    if constexpr (WIDE) gru_load<T, kGruVec>(p, v);
    else {
#pragma unroll
      for (int e = 0; e < kGruVec; ++e) v[e] = c + e < a.width ? to_f32(p[e]) : 0.f;
    }
  };
  // the tokens are dealt evenly: a portion shorter than a turn gives every thread fewer of them
  const int per = min(kGruTokens, (n + kGruRanks * kGruLanes - 1) / (kGruRanks * kGruLanes));
  for (int base = 0, turn = 0; base < n; base += kGruRanks * kGruLanes * per, turn ^= 1) {
    const int first = base + (rank * kGruLanes + tl) * per, last = live ? min(n, first + per) : first;
    float ca[kGruVec], cb[kGruVec];
#pragma unroll
    for (int e = 0; e < kGruVec; ++e) { ca[e] = 1.f; cb[e] = 0.f; }
#pragma unroll 4
    for (int t = first; t < last; ++t) {
      float z[kGruVec], u[kGruVec];
      load(a.z, t, z);
      load(a.u, t, u);
      asm volatile("prefetch.global.L2 [%0];" ::"l"((const T*)a.g + (size_t)(t0 + t) * a.stride + c));     // for the second walk
#pragma unroll
      for (int e = 0; e < kGruVec; ++e) {
        float m, b;
        gru_step(z[e] + bz[e], u[e] + bu[e], m, b);
        cb[e] = fmaf(m, cb[e], b);
        ca[e] *= m;
      }
    }
    gru_store<float, kGruVec>(&fa[tl][grp * kGruVec], ca);
    gru_store<float, kGruVec>(&fb[tl][grp * kGruVec], cb);
    __syncthreads();
    if (tid < kGruChannels) {                       // fold the lanes; each finds the composition of those before it
      float xa = 1.f, xb = 0.f;
#pragma unroll
      for (int l = 0; l < kGruLanes; ++l) {
        const float la = fa[l][tid], lb = fb[l][tid];
        fa[l][tid] = xa;
        fb[l][tid] = xb;
        xb = fmaf(la, xb, lb);
        xa *= la;
      }
      tot[turn][0][tid] = xa;
      tot[turn][1][tid] = xb;
    }
    cluster.sync();
    if (tid < kGruChannels) {                       // the state before this block's tokens, and after the whole turn
      float xa[kGruRanks], xb[kGruRanks];
#pragma unroll
      for (int r = 0; r < kGruRanks; ++r) {
        const float* remote = cluster.map_shared_rank(&tot[turn][0][0], r);
        xa[r] = remote[tid];
        xb[r] = remote[kGruChannels + tid];
      }
#pragma unroll
      for (int r = 0; r < kGruRanks; ++r) {
        if (r == rank) start[tid] = carry;
        carry = fmaf(xa[r], carry, xb[r]);
      }
    }
    __syncthreads();
    float S[kGruVec];
#pragma unroll
    for (int e = 0; e < kGruVec; ++e) {
      const int k = grp * kGruVec + e;
      S[e] = fmaf(fa[tl][k], start[k], fb[tl][k]);
    }
#pragma unroll 4
    for (int t = first; t < last; ++t) {
      float z[kGruVec], u[kGruVec], g[kGruVec], o[kGruVec];
      load(a.z, t, z);
      load(a.u, t, u);
      load(a.g, t, g);
#pragma unroll
      for (int e = 0; e < kGruVec; ++e) {
        float m, b;
        gru_step(z[e] + bz[e], u[e] + bu[e], m, b);
        S[e] = fmaf(m, S[e], b);
        o[e] = S[e] * (g[e] * gru_sigmoid(g[e]));
      }
      T* p = (T*)a.out + (size_t)(t0 + t) * a.out_stride + c;
      if constexpr (WIDE) gru_store<T, kGruVec>(p, o);
      else {
#pragma unroll
        for (int e = 0; e < kGruVec; ++e) if (c + e < a.width) p[e] = from_f32<T>(o[e]);
      }
    }
    __syncthreads();                                // fa, fb and start are free for the next turn
  }
  // every block has read the slot before the first turn's cluster barrier; no block may end while others read its `tot`
  if (rank == 0 && tid < kGruChannels && my_channel < a.width) slot[my_channel] = carry;
  cluster.sync();
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
  const dim3 grid(ceil_div(width, kGruChannels), n_seqs, kGruRanks);
  if (dtype == LMSF_F32) {
    if (wide) min_gru_scan_kernel<float, true><<<grid, kGruThreads, 0, s>>>(a);
    else min_gru_scan_kernel<float, false><<<grid, kGruThreads, 0, s>>>(a);
  } else {
    if (wide) min_gru_scan_kernel<bf16, true><<<grid, kGruThreads, 0, s>>>(a);
    else min_gru_scan_kernel<bf16, false><<<grid, kGruThreads, 0, s>>>(a);
  }
  return LMSF_LAUNCH_STATUS();
}
