// What lies between two branches of a block around a float32 residual stream, for norms that may take the mean off (layer norm),
// a branch that may be a pair, and a short filter over time behind the next norm:
//
//   b    = y                                        one branch, or
//   b    = m * (y1 / rms(y1) * p1 + y2 / rms(y2) * p2)          a pair of branches, each with its own norm
//   res <- res + N_post(b)                          (if there is a branch);  res <- res + vec (if given)
//   h    = N_next(res)                              (if asked for), rounded to the activation type
//   h   <- h + sum_j f[j] * (h of the tokens before, its own last)   for single tokens: the inputs before come from the
//                                                   request's state slot, which is rolled on
//   N(x) = (x - c) / sqrt(mean((x - c)^2) + eps) * w,  c the mean of x, or zero (a division by the root mean square)
//
// Every sum, root and product is float32; deviations are squared after the mean is taken off (two passes over registers).  One
// block per token; a row is read once and held in registers.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_layer_norm)

namespace lmsf {

constexpr int kThreads = 256;
constexpr int kFewRows = 296;        // up to two rows an SM: a block of 1,024 threads per row, a piece of the row each
constexpr int kMaxPerThread = 64;   // widths up to 16,384
constexpr int kMaxFilterTaps = 32;

struct StreamLayerArgs {
  float* res;
  const void* y1; const void* y2;                    // [n, hidden] of the activation type; either may be null (y2 needs y1)
  const float* p1; const float* p2; float pair_eps, pair_factor;
  const float* w_post; float eps_post; int post_centred;
  const float* vec;
  void* h; const float* w_next; float eps_next; int next_centred;
  const float* filter; int taps;                     // [taps][hidden]; null: none
  float* state; long long slot_stride; const int* state_slot;   // [taps - 1][hidden] per slot; token i is of request i
  int hidden;
};

template <int V> __device__ __forceinline__ void ldv(const float* p, float (&v)[V]) {
  if constexpr (V == 4) ld4(p, v); else v[0] = *p;
}
template <int V> __device__ __forceinline__ void ldv(const bf16* p, float (&v)[V]) {
  if constexpr (V == 4) ld4(p, v); else v[0] = __bfloat162float(*p);
}
template <int V, typename T> __device__ __forceinline__ void stv(T* p, const float (&v)[V]) {
  if constexpr (V == 4) st4(p, v); else *p = from_f32<T>(v[0]);
}

// Sums of two values over the block; every thread gets both.  `at` names one of the scratch rows: consecutive calls take
// different ones, so one barrier a call is enough.
template <int NW>
__device__ __forceinline__ float2 block_sum2(float a, float b, float2 (*scratch)[NW], int at) {
  a = warp_sum(a);
  b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) scratch[at][threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  if constexpr (NW <= 8) {
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < NW; ++w) { const float2 v = scratch[at][w]; s.x += v.x; s.y += v.y; }
    return s;
  } else {
    const float2 v = (threadIdx.x & 31) < NW ? scratch[at][threadIdx.x & 31] : make_float2(0.f, 0.f);
    return make_float2(warp_sum(v.x), warp_sum(v.y));
  }
}

// A vector of the model (a weight) at column i: read where it is used, or, in a build whose threads hold one piece of a row each,
// before anything of the step is waited for, so that its way from memory overlaps the kernel before this one.
template <int V> struct Early {
  float v[V];
  __device__ __forceinline__ void load(const float* p, int i, int D) { if (p != nullptr && i < D) ldv<V>(p + i, v); }
};

template <typename T, int PER, int V, int NT>
__global__ void __launch_bounds__(NT) stream_layer_kernel(const StreamLayerArgs a) {
  constexpr int NW = NT / 32;
  constexpr bool kEarly = PER == 1;
  constexpr int kEarlyTaps = 4;
  __shared__ float2 scratch[5][NW];
  const int D = a.hidden, tid = threadIdx.x;
  const size_t base = (size_t)blockIdx.x * D;
  const float inv_d = 1.0f / (float)D;
  auto at = [&](int it) { return (it * NT + tid) * V; };
  Early<V> e_p1, e_p2, e_post, e_vec, e_next, e_f[kEarlyTaps];
  pdl_launch_dependents();
  if constexpr (kEarly) {
    e_p1.load(a.p1, at(0), D);
    e_p2.load(a.p2, at(0), D);
    e_post.load(a.w_post, at(0), D);
    e_vec.load(a.vec, at(0), D);
    e_next.load(a.w_next, at(0), D);
#pragma unroll
    for (int j = 0; j < kEarlyTaps; ++j)
      if (a.filter != nullptr && j < a.taps) e_f[j].load(a.filter + (size_t)j * D, at(0), D);
  }
  auto weight = [&](const Early<V>& early, const float* p, int it, float (&w)[V]) {
    if constexpr (kEarly) {
#pragma unroll
      for (int e = 0; e < V; ++e) w[e] = early.v[e];
    } else {
      ldv<V>(p + at(it), w);
    }
  };
  pdl_wait();
  float* st = a.filter != nullptr && a.taps > 1 ? a.state + (size_t)a.state_slot[blockIdx.x] * a.slot_stride : nullptr;
  Early<V> e_st[kEarlyTaps - 1];                      // the carried inputs
  if constexpr (kEarly) {
#pragma unroll
    for (int j = 0; j < kEarlyTaps - 1; ++j)
      if (st != nullptr && j < a.taps - 1) e_st[j].load(st + (size_t)j * D, at(0), D);
  }
  float r[PER][V];
#pragma unroll
  for (int it = 0; it < PER; ++it) {
#pragma unroll
    for (int e = 0; e < V; ++e) r[it][e] = 0.f;
    if (at(it) < D) ldv<V>(a.res + base + at(it), r[it]);
  }
  if (a.y1 != nullptr) {
    float b[PER][V];
    float s1 = 0.f;
#pragma unroll
    for (int it = 0; it < PER; ++it) {
#pragma unroll
      for (int e = 0; e < V; ++e) b[it][e] = 0.f;
      if (at(it) < D) ldv<V>((const T*)a.y1 + base + at(it), b[it]);
    }
    if (a.y2 != nullptr) {
      float c[PER][V];
      float q1 = 0.f, q2 = 0.f;
#pragma unroll
      for (int it = 0; it < PER; ++it) {
#pragma unroll
        for (int e = 0; e < V; ++e) c[it][e] = 0.f;
        if (at(it) < D) ldv<V>((const T*)a.y2 + base + at(it), c[it]);
#pragma unroll
        for (int e = 0; e < V; ++e) { q1 = fmaf(b[it][e], b[it][e], q1); q2 = fmaf(c[it][e], c[it][e], q2); }
      }
      const float2 q = block_sum2<NW>(q1, q2, scratch, 0);
      const float i1 = a.pair_factor / sqrtf(fmaf(q.x, inv_d, a.pair_eps)), i2 = a.pair_factor / sqrtf(fmaf(q.y, inv_d, a.pair_eps));
#pragma unroll
      for (int it = 0; it < PER; ++it) {
        if (at(it) < D) {
          float w1[V], w2[V];
          weight(e_p1, a.p1, it, w1);
          weight(e_p2, a.p2, it, w2);
#pragma unroll
          for (int e = 0; e < V; ++e) b[it][e] = (b[it][e] * i1) * w1[e] + (c[it][e] * i2) * w2[e];
        }
      }
    }
    float mean = 0.f;
    if (a.post_centred) {
#pragma unroll
      for (int it = 0; it < PER; ++it)
#pragma unroll
        for (int e = 0; e < V; ++e) s1 += b[it][e];
      mean = block_sum2<NW>(s1, 0.f, scratch, 1).x * inv_d;
    }
    float q = 0.f;
#pragma unroll
    for (int it = 0; it < PER; ++it)
      if (at(it) < D)
#pragma unroll
        for (int e = 0; e < V; ++e) { b[it][e] -= mean; q = fmaf(b[it][e], b[it][e], q); }
    const float inv = 1.0f / sqrtf(fmaf(block_sum2<NW>(q, 0.f, scratch, 2).x, inv_d, a.eps_post));
#pragma unroll
    for (int it = 0; it < PER; ++it) {
      if (at(it) < D) {
        float w[V];
        weight(e_post, a.w_post, it, w);
#pragma unroll
        for (int e = 0; e < V; ++e) r[it][e] = fmaf(b[it][e] * inv, w[e], r[it][e]);
      }
    }
  }
  if (a.vec != nullptr) {
#pragma unroll
    for (int it = 0; it < PER; ++it) {
      if (at(it) < D) {
        float f[V];
        weight(e_vec, a.vec, it, f);
#pragma unroll
        for (int e = 0; e < V; ++e) r[it][e] += f[e];
      }
    }
  }
  if (a.y1 != nullptr || a.vec != nullptr) {
#pragma unroll
    for (int it = 0; it < PER; ++it)
      if (at(it) < D) stv<V>(a.res + base + at(it), r[it]);
  }
  if (a.h == nullptr) return;
  float mean = 0.f;
  if (a.next_centred) {
    float s = 0.f;
#pragma unroll
    for (int it = 0; it < PER; ++it)
#pragma unroll
      for (int e = 0; e < V; ++e) s += r[it][e];
    mean = block_sum2<NW>(s, 0.f, scratch, 3).x * inv_d;
  }
  float q = 0.f;
#pragma unroll
  for (int it = 0; it < PER; ++it)
    if (at(it) < D)
#pragma unroll
      for (int e = 0; e < V; ++e) { r[it][e] -= mean; q = fmaf(r[it][e], r[it][e], q); }
  const float inv = 1.0f / sqrtf(fmaf(block_sum2<NW>(q, 0.f, scratch, 4).x, inv_d, a.eps_next));
#pragma unroll
  for (int it = 0; it < PER; ++it) {
    const int i = at(it);
    if (i >= D) continue;
    float w[V], o[V];
    weight(e_next, a.w_next, it, w);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = (r[it][e] * inv) * w[e];
    if (a.filter != nullptr) {
      // the row is rounded to the activation type before the filter, as where the filter is a kernel of its own
      float acc[V], f[V], u[V];
#pragma unroll
      for (int e = 0; e < V; ++e) { o[e] = to_f32(from_f32<T>(o[e])); acc[e] = 0.f; }
      const int taps = a.taps;
      if (kEarly && taps <= kEarlyTaps) {
#pragma unroll
        for (int j = 0; j < kEarlyTaps - 1; ++j) {
          if (j < taps - 1) {
#pragma unroll
            for (int e = 0; e < V; ++e) acc[e] = fmaf(e_f[j].v[e], e_st[j].v[e], acc[e]);
            if (j > 0) stv<V>(st + (size_t)(j - 1) * D + i, e_st[j].v);
          }
        }
#pragma unroll
        for (int j = 0; j < kEarlyTaps; ++j)
          if (j == taps - 1)
#pragma unroll
            for (int e = 0; e < V; ++e) f[e] = e_f[j].v[e];
      } else {
        for (int j = 0; j < taps - 1; ++j) {
          ldv<V>(st + (size_t)j * D + i, u);
          ldv<V>(a.filter + (size_t)j * D + i, f);
#pragma unroll
          for (int e = 0; e < V; ++e) acc[e] = fmaf(f[e], u[e], acc[e]);
          if (j > 0) stv<V>(st + (size_t)(j - 1) * D + i, u);
        }
        ldv<V>(a.filter + (size_t)(taps - 1) * D + i, f);
      }
      if (taps > 1) stv<V>(st + (size_t)(taps - 2) * D + i, o);
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] += fmaf(f[e], o[e], acc[e]);
    }
    stv<V>((T*)a.h + base + i, o);
  }
}

template <typename T>
static int pick_stream_layer(const StreamLayerArgs& a, int n, cudaStream_t s) {
  const bool wide = a.hidden % 4 == 0 && ((uintptr_t)a.res | (uintptr_t)a.p1 | (uintptr_t)a.p2 | (uintptr_t)a.w_post | (uintptr_t)a.vec |
                                          (uintptr_t)a.w_next | (uintptr_t)a.filter | (uintptr_t)a.state) % 16 == 0 && a.slot_stride % 4 == 0 &&
                    ((uintptr_t)a.y1 | (uintptr_t)a.y2 | (uintptr_t)a.h) % (4 * sizeof(T)) == 0;
  const int per = ceil_div(a.hidden, kThreads * (wide ? 4 : 1));
  if (wide && per > 1 && per <= 4 && n <= kFewRows) return launch_pdl(stream_layer_kernel<T, 1, 4, 1024>, dim3(n), dim3(1024), 0, s, a);
#define LMSF_GO(P, V) return launch_pdl(stream_layer_kernel<T, P, V, kThreads>, dim3(n), dim3(kThreads), 0, s, a)
#define LMSF_CASE(P) if (per <= P) { if (wide) LMSF_GO(P, 4); else LMSF_GO(P, 1); }
  LMSF_CASE(1) LMSF_CASE(2) LMSF_CASE(4) LMSF_CASE(8) LMSF_CASE(16)
  if (!wide) { if (per <= 32) LMSF_GO(32, 1); LMSF_GO(64, 1); }
#undef LMSF_CASE
#undef LMSF_GO
  return LMSF_EBADARG;
}

}  // namespace lmsf

// res: float32 [n, hidden].  y1, y2 (a pair, with its norms' weights p1, p2), h: [n, hidden] of `dtype`; weights, vec: float32
// [hidden].  With `filter` (float32 [taps, hidden]) every row is the single token of a request: row i belongs to the slot
// state_slot[i], whose [taps - 1, hidden] floats start at state + slot * slot_stride.
LMSF_API int lmsf_stream_layer(float* res, const void* y1, const void* y2, const float* p1, const float* p2, float pair_eps,
                               float pair_factor, const float* w_post, float eps_post, int post_centred, const float* vec, void* h,
                               const float* w_next, float eps_next, int next_centred, const float* filter, int taps, float* state,
                               long long slot_stride, const int* state_slot, int n, int hidden, int dtype, void* stream) {
  using namespace lmsf;
  if (n <= 0) return 0;
  if (hidden <= 0 || hidden > kThreads * kMaxPerThread) LMSF_REFUSE("stream_layer: width %d is outside 1..%d", hidden, kThreads * kMaxPerThread);
  if (y1 && (!w_post || !(eps_post > 0.f))) LMSF_REFUSE("stream_layer: a branch needs the weight of its norm and a positive eps");
  if (y2 && (!y1 || !p1 || !p2 || !(pair_eps > 0.f))) LMSF_REFUSE("stream_layer: a pair needs both branches, both weights and a positive eps");
  if (h && (!w_next || !(eps_next > 0.f))) LMSF_REFUSE("stream_layer: the next norm needs its weight and a positive eps");
  if (filter && (!h || taps < 1 || taps > kMaxFilterTaps || !state_slot || (taps > 1 && !state)))
    LMSF_REFUSE("stream_layer: a filter of %d taps (1 to %d) needs a next norm, its state and the slots", taps, kMaxFilterTaps);
  StreamLayerArgs a{res, y1, y2, p1, p2, pair_eps, pair_factor, w_post, eps_post, post_centred ? 1 : 0, vec, h, w_next, eps_next,
                    next_centred ? 1 : 0, filter, taps, state, slot_stride, state_slot, hidden};
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == LMSF_F32) return pick_stream_layer<float>(a, n, s);
  if (dtype == LMSF_BF16) return pick_stream_layer<bf16>(a, n, s);
  LMSF_REFUSE("stream_layer: unknown dtype code %d", dtype);
}
