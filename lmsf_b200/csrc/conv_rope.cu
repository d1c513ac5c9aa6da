// Queries and keys that pass a short causal filter over time on their way into attention, in one kernel behind the projection:
//
//   y[t, c] = sum_j w[j, c] * u[t - (taps - 1) + j, c]        u: the projection's columns of q and k, bias included
//   q[t]    = turned(y of the query heads)                     to a matrix of its own
//   page    : key plane = turned(y of the key heads), value plane = y of the key heads as they are
//
// Inputs before a portion's first token come from the request's state slot ([taps - 1, channels] float32), which is rolled on.
// Of a head's first rot_dim values, i and i + rot_dim / 2 turn by position * inv_freq[i], cos and sin times a constant; the rest
// passes.  The filter, the angles and the rotation are float32; a value is rounded once, where it is stored.
//
// A thread owns 2 V channels of a head for a chunk of tokens: V values and the V they are paired with (or, in the part that is not
// turned, V values and the V half that part further on), so a turned pair never leaves its thread; the window of taps - 1 inputs
// slides in registers.  The thread of a request's first chunk is the only reader and writer of its channels' state.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_conv_rope)

namespace lmsf {

constexpr int kThreads = 128;
#ifndef LMSF_ROPE_CHUNK
#define LMSF_ROPE_CHUNK 8
#endif
constexpr int kChunk = LMSF_ROPE_CHUNK;   // tokens per block
constexpr int kMaxTaps = 32;

struct ConvRopeArgs {
  const void* x; long long x_stride;           // [n, (n_q_heads + n_kv_heads) * hd]
  void* q; long long q_stride;                 // [n, n_q_heads * hd]
  const float* w; int taps;                    // [taps][channels]
  float* state; long long slot_stride;         // [taps - 1][channels] of slot s at state + s * slot_stride
  const int* cu_q; const int* state_slot; const int* positions;
  const int* block_table; int max_blocks, block_size;
  void* cache; long long page_stride;          // [page][2][n_kv_heads][slot][hd]
  const float* inv_freq; int rot_dim; float mult;   // inv_freq null: nothing is turned
  int n_q_heads, n_kv_heads, hd;
  int* error_flag;
};

template <int V> __device__ __forceinline__ void ld_vals(const float* p, float* v) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) { const float4 a = *reinterpret_cast<const float4*>(p + i); v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w; }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = p[i];
  }
}
template <int V> __device__ __forceinline__ void ld_vals(const bf16* p, float* v) {
  if constexpr (V == 8) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
#pragma unroll
    for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  } else if constexpr (V == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
#pragma unroll
    for (int i = 0; i < 2; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = __bfloat162float(p[i]);
  }
}
template <int V> __device__ __forceinline__ void st_vals(float* p, const float* v) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = v[i];
  }
}
template <int V> __device__ __forceinline__ void st_vals(bf16* p, const float* v) {
  if constexpr (V == 8) {
    uint4 a;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&a);
#pragma unroll
    for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = a;
  } else if constexpr (V == 4) {
    uint2 a;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&a);
#pragma unroll
    for (int i = 0; i < 2; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint2*>(p) = a;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16_rn(v[i]);
  }
}

// V consecutive values in the stored type, moved in one access
template <typename T, int V> struct alignas(sizeof(T) * V) Piece { T v[V]; };
constexpr int kAhead = 4;

// TAPS 0: any number of taps, inputs read again for every token, one block for a whole portion (a chunk may be shorter than the
// filter, so only the block that rolls the state on may read it).
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(kThreads) conv_rope_kernel(const ConvRopeArgs a) {
  extern __shared__ float cs[];                // [token of the chunk][cos: half | sin: half]
  __shared__ long long row_off[kChunk];        // the token's row inside the cache, kv head 0; negative: no page
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z;
  int lo = blockIdx.y * kChunk;
  const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
  if (lo >= n) return;
  int cnt = min(kChunk, n - lo);
  const int half = a.inv_freq ? a.rot_dim / 2 : 0;
  auto stage = [&]() {                         // angles and pages of the chunk's tokens, by the whole block
    for (int i = threadIdx.x; i < cnt * half; i += kThreads) {
      const int t = i / half, p = i % half;
      float s, c;
      sincosf((float)a.positions[t0 + lo + t] * a.inv_freq[p], &s, &c);
      cs[t * 2 * half + p] = c * a.mult;
      cs[t * 2 * half + half + p] = s * a.mult;
    }
    if (threadIdx.x < cnt) {
      const int pos = a.positions[t0 + lo + threadIdx.x];
      const int page = a.block_table[(size_t)seq * a.max_blocks + pos / a.block_size];
      if (page < 0 && blockIdx.x == 0 && a.error_flag) atomicExch(a.error_flag, 2);
      row_off[threadIdx.x] = page < 0 ? -1 : (long long)page * a.page_stride + (long long)(pos % a.block_size) * a.hd;
    }
    __syncthreads();
  };
  stage();
  const int per_head = a.hd / (2 * V), heads = a.n_q_heads + a.n_kv_heads;
  int item = blockIdx.x * kThreads + threadIdx.x;
  const bool live = item < per_head * heads;
  if (TAPS > 0 && !live) return;
  if (!live) item = 0;                         // (TAPS 0: keeps the block's barriers)
  const int head = item / per_head, w = item % per_head;
  const bool turned = w * V < half;            // the first half / V items of a head
  const int tail = a.hd - 2 * half;
  const int i0 = turned ? w * V : 2 * half + (w * V - half);
  const int i1 = turned ? i0 + half : i0 + tail / 2;
  const int C = heads * a.hd, c0 = head * a.hd + i0, c1 = head * a.hd + i1;
  const T* __restrict__ x = (const T*)a.x + (size_t)t0 * a.x_stride;
  float* st = a.taps > 1 ? a.state + (size_t)a.state_slot[seq] * a.slot_stride : nullptr;
  const bool is_q = head < a.n_q_heads;
  T* qo = (T*)a.q + (size_t)t0 * a.q_stride + c0;
  T* ko = (T*)a.cache + (size_t)(head - a.n_q_heads) * a.block_size * a.hd;
  const long long v_off = (long long)a.n_kv_heads * a.block_size * a.hd;

  auto emit = [&](int t, const float (&y)[2 * V]) {       // t: token of the portion
    float z[2 * V];
    if (turned) {
      const float* c = cs + (t - lo) * 2 * half + i0;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        z[e] = y[e] * c[e] - y[V + e] * c[half + e];
        z[V + e] = y[V + e] * c[e] + y[e] * c[half + e];
      }
    } else {
#pragma unroll
      for (int e = 0; e < 2 * V; ++e) z[e] = y[e];
    }
    if (is_q) {
      T* o = qo + (size_t)t * a.q_stride;
      st_vals<V>(o, z);
      st_vals<V>(o + (i1 - i0), z + V);
    } else {
      const long long r = row_off[t - lo];
      if (r < 0) return;
      T* k = ko + r;
      st_vals<V>(k + i0, z);
      st_vals<V>(k + i1, z + V);
      st_vals<V>(k + v_off + i0, y);
      st_vals<V>(k + v_off + i1, y + V);
    }
  };
  // input u of this thread's channels (negative: before the portion), as floats
  const int taps = TAPS ? TAPS : a.taps;
  auto input = [&](int u, float (&v)[2 * V]) {
    if (u >= 0) {
      const T* p = x + (size_t)u * a.x_stride;
      ld_vals<V>(p + c0, v);
      ld_vals<V>(p + c1, v + V);
    } else {
      const float* p = st + (size_t)(taps - 1 + u) * C;
      ld_vals<V>(p + c0, v);
      ld_vals<V>(p + c1, v + V);
    }
  };
  if constexpr (TAPS > 0) {
    float wr[TAPS][2 * V], win[TAPS > 1 ? TAPS - 1 : 1][2 * V];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      ld_vals<V>(a.w + (size_t)j * C + c0, wr[j]);
      ld_vals<V>(a.w + (size_t)j * C + c1, wr[j] + V);
    }
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) input(lo - (TAPS - 1) + j, win[j]);
    // four tokens' inputs are asked for together, in the stored type
    for (int tb = lo; tb < lo + cnt; tb += kAhead) {
      Piece<T, V> in[kAhead][2];
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        if (tb + u < lo + cnt) {
          const T* p = x + (size_t)(tb + u) * a.x_stride;
          in[u][0] = *reinterpret_cast<const Piece<T, V>*>(p + c0);
          in[u][1] = *reinterpret_cast<const Piece<T, V>*>(p + c1);
        }
      }
#pragma unroll
      for (int u = 0; u < kAhead; ++u) {
        if (tb + u >= lo + cnt) break;
        float cur[2 * V], y[2 * V];
        ld_vals<V>(in[u][0].v, cur);
        ld_vals<V>(in[u][1].v, cur + V);
#pragma unroll
        for (int e = 0; e < 2 * V; ++e) {
          float s = 0.f;
#pragma unroll
          for (int j = 0; j < TAPS - 1; ++j) s = fmaf(wr[j][e], win[j][e], s);
          y[e] = fmaf(wr[TAPS - 1][e], cur[e], s);
#pragma unroll
          for (int j = 0; j + 1 < TAPS - 1; ++j) win[j][e] = win[j + 1][e];
          if (TAPS > 1) win[TAPS > 1 ? TAPS - 2 : 0][e] = cur[e];
        }
        emit(tb + u, y);
      }
    }
    if (lo != 0 || TAPS == 1) return;
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      float v[2 * V];
      if (n > kChunk) input(n - (TAPS - 1) + j, v);       // the portion's last inputs (n > taps - 1); else the window holds them
      else {
#pragma unroll
        for (int e = 0; e < 2 * V; ++e) v[e] = win[j][e];
      }
      st_vals<V>(st + (size_t)j * C + c0, v);
      st_vals<V>(st + (size_t)j * C + c1, v + V);
    }
  } else {
    while (true) {
      for (int t = lo; live && t < lo + cnt; ++t) {
        float y[2 * V], v[2 * V], wj[2 * V];
#pragma unroll
        for (int e = 0; e < 2 * V; ++e) y[e] = 0.f;
        for (int j = 0; j < taps; ++j) {
          input(t - (taps - 1) + j, v);
          ld_vals<V>(a.w + (size_t)j * C + c0, wj);
          ld_vals<V>(a.w + (size_t)j * C + c1, wj + V);
#pragma unroll
          for (int e = 0; e < 2 * V; ++e) y[e] = fmaf(wj[e], v[e], y[e]);
        }
        emit(t, y);
      }
      lo += kChunk;
      if (lo >= n) break;
      cnt = min(kChunk, n - lo);
      __syncthreads();                         // the chunk before has been read
      stage();
    }
    if (!live) return;
    for (int j = 0; j < taps - 1; ++j) {                   // row j takes input n - (taps - 1) + j: a later row, or the portion
      float v[2 * V];
      input(n - (taps - 1) + j, v);
      st_vals<V>(st + (size_t)j * C + c0, v);
      st_vals<V>(st + (size_t)j * C + c1, v + V);
    }
  }
}

template <typename T, int V>
static int launch_conv_rope(const ConvRopeArgs& a, int n_seqs, int max_q, cudaStream_t s) {
  dim3 grid(ceil_div((a.n_q_heads + a.n_kv_heads) * (a.hd / (2 * V)), kThreads), ceil_div(max_q, kChunk), n_seqs);
  const size_t smem = a.inv_freq ? (size_t)kChunk * a.rot_dim * sizeof(float) : 0;
#define LMSF_CASE(N) case N: return launch_pdl(conv_rope_kernel<T, V, N>, grid, dim3(kThreads), smem, s, a)
  switch (a.taps) { LMSF_CASE(1); LMSF_CASE(2); LMSF_CASE(3); LMSF_CASE(4); default: break; }
#undef LMSF_CASE
  grid.y = 1;
  return launch_pdl(conv_rope_kernel<T, V, 0>, grid, dim3(kThreads), smem, s, a);
}

}  // namespace lmsf

// x: [n, (n_q_heads + n_kv_heads) * head_dim] of `dtype` (queries, then keys); q: [n, n_q_heads * head_dim]; w: float32
// [taps][channels]; state: see above; cache: [page][2][n_kv_heads][block_size][head_dim].  max_q: the longest portion (sizes the
// grid only).  head_dim and rot_dim are even; rot_dim up to 512.
LMSF_API int lmsf_conv_rope_cache(const void* x, long long x_stride, void* q, long long q_stride, const float* w, int taps, float* state,
                                  long long slot_stride, const int* cu_q, const int* state_slot, const int* positions,
                                  const int* block_table, int max_blocks, int block_size, void* cache, long long page_stride,
                                  const float* inv_freq, int rot_dim, float mult, int n_q_heads, int n_kv_heads, int head_dim, int n_seqs,
                                  int max_q, int dtype, int* error_flag, void* stream) {
  using namespace lmsf;
  if (n_seqs <= 0 || max_q <= 0) return 0;
  if (taps < 1 || taps > kMaxTaps) LMSF_REFUSE("conv_rope: %d taps (1 to %d)", taps, kMaxTaps);
  if (n_q_heads <= 0 || n_kv_heads <= 0 || head_dim <= 0 || head_dim % 2) LMSF_REFUSE("conv_rope: %d + %d heads of %d", n_q_heads, n_kv_heads, head_dim);
  if (inv_freq && (rot_dim <= 0 || rot_dim % 2 || rot_dim > head_dim || rot_dim > 512))
    LMSF_REFUSE("conv_rope: rot_dim=%d must be even and at most head_dim=%d", rot_dim, head_dim);
  if (block_size <= 0 || max_blocks <= 0 || !cache || !block_table || (taps > 1 && !state)) LMSF_REFUSE("conv_rope: a cache, its block table and the state are needed");
  if (n_seqs > 65535 || ceil_div(max_q, kChunk) > 65535) LMSF_REFUSE("conv_rope: too many requests or too long a portion for one launch");
  ConvRopeArgs a{x, x_stride, q, q_stride, w, taps, state, slot_stride, cu_q, state_slot, positions, block_table, max_blocks, block_size,
                 cache, page_stride, inv_freq, rot_dim, mult, n_q_heads, n_kv_heads, head_dim, error_flag};
  cudaStream_t s = (cudaStream_t)stream;
  const int half = inv_freq ? rot_dim / 2 : 0, tail = head_dim - 2 * half, C = (n_q_heads + n_kv_heads) * head_dim;
  const int esz = dtype == LMSF_F32 ? 4 : 2;
  auto takes = [&](int v) {
    return half % v == 0 && tail % (2 * v) == 0 && x_stride % v == 0 && q_stride % v == 0 && page_stride % v == 0 && C % 4 == 0 &&
           slot_stride % 4 == 0 && ((uintptr_t)w | (uintptr_t)state) % 16 == 0 &&
           ((uintptr_t)x | (uintptr_t)q | (uintptr_t)cache) % (v * esz) == 0;
  };
  if (dtype == LMSF_F32) return takes(4) ? launch_conv_rope<float, 4>(a, n_seqs, max_q, s) : launch_conv_rope<float, 1>(a, n_seqs, max_q, s);
  if (dtype != LMSF_BF16) LMSF_REFUSE("conv_rope: unknown dtype code %d", dtype);
  if (takes(8)) return launch_conv_rope<bf16, 8>(a, n_seqs, max_q, s);
  if (takes(4)) return launch_conv_rope<bf16, 4>(a, n_seqs, max_q, s);
  return launch_conv_rope<bf16, 1>(a, n_seqs, max_q, s);
}
