// A matrix memory with exponential gates (the mLSTM cell of xLSTM): per request and head a matrix S [dk, dv], a vector n
// [dk] and a running maximum m, all float32, kept across steps in a state slot.
//
//   i = cap tanh((raw_i + b_i) / cap),  f = log sigmoid(cap tanh((raw_f + b_f) / cap))
//   m_t = max(f + m_(t-1), i);  keep = exp(f + m_(t-1) - m_t);  write = exp(i - m_t)
//   S_t = keep S_(t-1) + write k v^T;  n_t = keep n_(t-1) + write k
//   o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + eps)                     (q times a constant; m starts at 0)
//
// q, k, v and the two gate logits arrive as columns of a projection's output.  Everything behind them is float32.
//
// Two ways through a portion of tokens:
//   * single tokens and short portions: memory_scan_kernel, one block per (request, head, 64 value columns), token by token.
//     Warp w holds rows [w R, (w + 1) R) of the block's 64 columns in registers, two columns per lane; tokens are staged in
//     chunks; the warps' partial outputs are added up in shared memory in a fixed order.  A decode step reads and writes the
//     state once.
//   * long portions: chunks of 64 tokens in three launches.  With F the sum of f from the chunk's start (kept in double, so
//     that differences of large sums stay exact), token s adds exp(F_end - F_s + i_s) k_s v_s^T to the state at the chunk's
//     end and exp(F_t - F_s + i_s) (q_t . k_s) v_s to the output of token t >= s:
//       memory_chunk_kernel   per chunk: what it adds to the state (in tiles of 64 x 64) and its score matrix with the gates
//                             applied, each scaled by its own maximum
//       memory_prefix_kernel  walks every portion's chunks in order: the state before each chunk, the state in the slot
//       memory_output_kernel  per chunk and 64 value columns: one product [q | scores] x [state before; v], then the division
//
// A slot holds [heads][dk][dv] of S, then for every tile of 64 value columns a copy of n [heads][dk], then for every tile a
// copy of m [heads]: each block reads and writes the copy of its own tile, so no block waits for another.
#include "common.cuh"

LMSF_DEFINE_LAST_ERROR(lmsf_matrix_memory)

namespace lmsf {

constexpr int kWarps = 4;
constexpr int kMaxDk = 256;
constexpr int kCols = 64;      // value columns of the state per block
constexpr int kChunkTokens = 64;

struct MemoryArgs {
  const void* q; const void* k; const void* v;      // rows of [n_tokens, *]; head h starts at h * dk (q, k) or h * dv (v)
  long long q_stride, k_stride, v_stride;
  const void* gi; const void* gf; long long g_stride;   // [n_tokens, heads] gate logits
  const float* bi; const float* bf;                 // [heads]
  float cap, q_scale, eps;
  float* out; long long out_stride;                 // [n_tokens, heads * dv] float32
  float* state; long long slot_stride;
  const int* cu_q; const int* state_slot;
  int heads, dk, dv;
  const int4* items;                                // (request, first token, end token, chunk index); null: item i is request i, whole
  // long portions: per chunk and head
  float* added;                                     // [dk][dv] and [dk]: what the chunk adds; then the state before it
  float* scores;                                    // [64 s][64 t]
  float* rows;                                      // [3][64]: F_t, the scores' maximum and the sum of a token's scores
  float* ends;                                      // [2]: F at the chunk's end, the maximum that `added` is scaled by
  float* m_before;                                  // [1]
};

__device__ __forceinline__ long long n_offset(const MemoryArgs& a, int tile) {
  return ((long long)a.heads * a.dk) * a.dv + (long long)tile * a.heads * a.dk;
}
__device__ __forceinline__ long long m_offset(const MemoryArgs& a, int tile) {
  const int tiles = (a.dv + kCols - 1) / kCols;
  return ((long long)a.heads * a.dk) * (a.dv + tiles) + (long long)tile * a.heads;
}
__device__ __forceinline__ float log_input_gate(const MemoryArgs& a, float raw, int head) {
  return a.cap * tanhf((raw + a.bi[head]) / a.cap);
}
__device__ __forceinline__ float log_forget_gate(const MemoryArgs& a, float raw, int head) {
  const float z = a.cap * tanhf((raw + a.bf[head]) / a.cap);
  return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// ------------------------------------------------------------------------------------------------ token by token
template <typename T, int R>
__global__ void __launch_bounds__(kWarps * 32) memory_scan_kernel(MemoryArgs a) {
  constexpr int kRows = kWarps * R;                  // rows of the state that the block walks (>= dk; the rest are zeros)
  constexpr int kChunk = R > 32 ? 8 : 16;            // tokens staged at a time
  constexpr int kN = (R + 31) / 32;                  // values of n per lane
  __shared__ __align__(16) float qs[kChunk][kRows];
  __shared__ __align__(16) float ks[kChunk][kRows];
  __shared__ __align__(16) float vs[kChunk][kCols];
  __shared__ float part[kWarps][kChunk][kCols];
  __shared__ float part_n[kChunk][kWarps * 32];
  __shared__ float s_keep[kChunk], s_write[kChunk], s_floor[kChunk], s_den[kChunk];
  __shared__ float s_m;
  pdl_launch_dependents();
  const int head = blockIdx.y, tile = blockIdx.z, col0 = tile * kCols;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  pdl_wait();
  int seq = blockIdx.x, t0, t1;
  if (a.items != nullptr) {
    const int4 it = a.items[blockIdx.x];
    seq = it.x; t0 = it.y; t1 = it.z;
  } else {
    t0 = a.cu_q[seq]; t1 = a.cu_q[seq + 1];
  }
  if (t1 <= t0) return;
  const int dk = a.dk, dv = a.dv;
  const int cA = col0 + lane, cB = col0 + 32 + lane;
  const bool liveA = cA < dv, liveB = cB < dv;
  float* slot = a.state + (size_t)a.state_slot[seq] * a.slot_stride;
  float* st = slot + ((size_t)head * dk) * dv;
  float* nn = slot + n_offset(a, tile) + (size_t)head * dk;
  float* mm = slot + m_offset(a, tile) + head;
  const int r0 = warp * R;
  float SA[R], SB[R], N[kN];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    SA[i] = (liveA && r0 + i < dk) ? st[(size_t)(r0 + i) * dv + cA] : 0.f;
    SB[i] = (liveB && r0 + i < dk) ? st[(size_t)(r0 + i) * dv + cB] : 0.f;
  }
#pragma unroll
  for (int j = 0; j < kN; ++j) {
    const int i = lane + 32 * j;
    N[j] = (i < R && r0 + i < dk) ? nn[r0 + i] : 0.f;
  }
  if (threadIdx.x == 0) s_m = *mm;
  const T* qg = (const T*)a.q + (size_t)head * dk;
  const T* kg = (const T*)a.k + (size_t)head * dk;
  const T* vg = (const T*)a.v + (size_t)head * dv + col0;
  const bool wide_qk = dk % 4 == 0 && a.q_stride % 4 == 0 && a.k_stride % 4 == 0 && ((uintptr_t)a.q | (uintptr_t)a.k) % (4 * sizeof(T)) == 0;
  const bool wide_v = dv % 4 == 0 && a.v_stride % 4 == 0 && (uintptr_t)a.v % (4 * sizeof(T)) == 0;

  for (int c0 = t0; c0 < t1; c0 += kChunk) {
    const int n = min(kChunk, t1 - c0);
    __syncthreads();   // the chunk before has been read
    if (wide_qk) {
      for (int e = threadIdx.x; e < n * (kRows / 4); e += kWarps * 32) {
        const int t = e / (kRows / 4), d = (e - t * (kRows / 4)) * 4;
        float kk[4] = {0.f, 0.f, 0.f, 0.f}, qq[4] = {0.f, 0.f, 0.f, 0.f};
        if (d < dk) {
          ld4(kg + (size_t)(c0 + t) * a.k_stride + d, kk);
          ld4(qg + (size_t)(c0 + t) * a.q_stride + d, qq);
#pragma unroll
          for (int u = 0; u < 4; ++u) qq[u] *= a.q_scale;
        }
        st4(&ks[t][d], kk);
        st4(&qs[t][d], qq);
      }
    } else {
      for (int e = threadIdx.x; e < n * kRows; e += kWarps * 32) {
        const int t = e / kRows, d = e - t * kRows;
        qs[t][d] = d < dk ? to_f32(qg[(size_t)(c0 + t) * a.q_stride + d]) * a.q_scale : 0.f;
        ks[t][d] = d < dk ? to_f32(kg[(size_t)(c0 + t) * a.k_stride + d]) : 0.f;
      }
    }
    if (wide_v) {
      for (int e = threadIdx.x; e < n * (kCols / 4); e += kWarps * 32) {
        const int t = e / (kCols / 4), c = (e - t * (kCols / 4)) * 4;
        float vv[4] = {0.f, 0.f, 0.f, 0.f};
        if (col0 + c < dv) ld4(vg + (size_t)(c0 + t) * a.v_stride + c, vv);
        st4(&vs[t][c], vv);
      }
    } else {
      for (int e = threadIdx.x; e < n * kCols; e += kWarps * 32) {
        const int t = e / kCols, c = e - t * kCols;
        vs[t][c] = col0 + c < dv ? to_f32(vg[(size_t)(c0 + t) * a.v_stride + c]) : 0.f;
      }
    }
    if (warp == kWarps - 1) {
      // the chunk's gates: one token a lane, then the running maximum by a scan over (f, i) pairs, m -> max(m + f, i)
      float f = 0.f, i = -INFINITY;
      if (lane < n) {
        i = log_input_gate(a, to_f32(((const T*)a.gi)[(size_t)(c0 + lane) * a.g_stride + head]), head);
        f = log_forget_gate(a, to_f32(((const T*)a.gf)[(size_t)(c0 + lane) * a.g_stride + head]), head);
      }
      float F = f, I = i;
#pragma unroll
      for (int off = 1; off < kChunk; off <<= 1) {
        const float Fp = __shfl_up_sync(0xffffffffu, F, off), Ip = __shfl_up_sync(0xffffffffu, I, off);
        if (lane >= off) { I = fmaxf(Ip + F, I); F += Fp; }
      }
      const float m_start = s_m;
      const float m = fmaxf(m_start + F, I);
      const float m_up = __shfl_up_sync(0xffffffffu, m, 1);
      const float m_prev = lane == 0 ? m_start : m_up;
      if (lane < n) {
        s_keep[lane] = expf(f + m_prev - m);
        s_write[lane] = expf(i - m);
        s_floor[lane] = expf(-m);
      }
      __syncwarp();
      if (lane == n - 1) s_m = m;
    }
    __syncthreads();
    for (int t = 0; t < n; ++t) {
      const float keep = s_keep[t], write = s_write[t];
      const float vA = write * vs[t][lane], vB = write * vs[t][32 + lane];
      float oA = 0.f, oB = 0.f, on = 0.f;
      const float4* k4 = reinterpret_cast<const float4*>(&ks[t][r0]);
      const float4* q4 = reinterpret_cast<const float4*>(&qs[t][r0]);
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const float4 kk = k4[i], qq = q4[i];
        SA[4 * i + 0] = fmaf(keep, SA[4 * i + 0], kk.x * vA);  SB[4 * i + 0] = fmaf(keep, SB[4 * i + 0], kk.x * vB);
        SA[4 * i + 1] = fmaf(keep, SA[4 * i + 1], kk.y * vA);  SB[4 * i + 1] = fmaf(keep, SB[4 * i + 1], kk.y * vB);
        SA[4 * i + 2] = fmaf(keep, SA[4 * i + 2], kk.z * vA);  SB[4 * i + 2] = fmaf(keep, SB[4 * i + 2], kk.z * vB);
        SA[4 * i + 3] = fmaf(keep, SA[4 * i + 3], kk.w * vA);  SB[4 * i + 3] = fmaf(keep, SB[4 * i + 3], kk.w * vB);
        oA = fmaf(qq.x, SA[4 * i + 0], oA);  oB = fmaf(qq.x, SB[4 * i + 0], oB);
        oA = fmaf(qq.y, SA[4 * i + 1], oA);  oB = fmaf(qq.y, SB[4 * i + 1], oB);
        oA = fmaf(qq.z, SA[4 * i + 2], oA);  oB = fmaf(qq.z, SB[4 * i + 2], oB);
        oA = fmaf(qq.w, SA[4 * i + 3], oA);  oB = fmaf(qq.w, SB[4 * i + 3], oB);
      }
#pragma unroll
      for (int j = 0; j < kN; ++j) {
        const int i = lane + 32 * j;
        if (i < R) {
          N[j] = fmaf(keep, N[j], write * ks[t][r0 + i]);
          on = fmaf(qs[t][r0 + i], N[j], on);
        }
      }
      part[warp][t][lane] = oA;
      part[warp][t][32 + lane] = oB;
      part_n[t][threadIdx.x] = on;
    }
    __syncthreads();
    for (int t = warp; t < n; t += kWarps) {           // a warp per token: n . q and the division's other side
      float s = 0.f;
#pragma unroll
      for (int w = 0; w < kWarps; ++w) s += part_n[t][w * 32 + lane];
      s = warp_sum(s);
      if (lane == 0) s_den[t] = fmaxf(fabsf(s), s_floor[t]) + a.eps;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n * kCols; e += kWarps * 32) {
      const int t = e / kCols, l = e - t * kCols;
      if (col0 + l < dv) {
        float o = part[0][t][l];
#pragma unroll
        for (int w = 1; w < kWarps; ++w) o += part[w][t][l];
        a.out[(size_t)(c0 + t) * a.out_stride + (size_t)head * dv + col0 + l] = o / s_den[t];
      }
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    if (liveA && r0 + i < dk) st[(size_t)(r0 + i) * dv + cA] = SA[i];
    if (liveB && r0 + i < dk) st[(size_t)(r0 + i) * dv + cB] = SB[i];
  }
#pragma unroll
  for (int j = 0; j < kN; ++j) {
    const int i = lane + 32 * j;
    if (i < R && r0 + i < dk) nn[r0 + i] = N[j];
  }
  if (threadIdx.x == 0) *mm = s_m;       // written before the chunk's last barrier, read by one thread only
}

// ------------------------------------------------------------------------------------------------ chunks of 64 tokens
constexpr int kPad = 68;               // floats of a staged row: 16-byte aligned, neighbouring rows on other banks
constexpr int kDepth = 32;             // inner dimension staged at a time
constexpr int kTileThreads = 256;      // 16 x 16 threads, 4 x 4 results each

// the chunk's gates by the first 64 threads; every thread of the block calls it.  sF: sum of f up to and with a token (double),
// sI: log input gate (minus infinity behind the chunk's end)
template <typename T>
__device__ __forceinline__ void chunk_gates(const MemoryArgs& a, int t0, int n, int head, double* sF, float* sI, double* carry) {
  const int t = threadIdx.x, lane = t & 31;
  double F = 0.0;
  if (t < kChunkTokens) {
    float i = -INFINITY;
    if (t < n) {
      i = log_input_gate(a, to_f32(((const T*)a.gi)[(size_t)(t0 + t) * a.g_stride + head]), head);
      F = (double)log_forget_gate(a, to_f32(((const T*)a.gf)[(size_t)(t0 + t) * a.g_stride + head]), head);
    }
    sI[t] = i;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, F, off);
      if (lane >= off) F += p;
    }
    if (t == 31) *carry = F;
  }
  __syncthreads();
  if (t < kChunkTokens) sF[t] = t >= 32 ? F + *carry : F;
  __syncthreads();
}

// rows [0, n) x columns [d0, d0 + kDepth) of a head's matrix, transposed into dst[column][row], times `scale`
template <typename T>
__device__ __forceinline__ void stage_transposed(float (*dst)[kPad], const T* __restrict__ src, long long stride, int n, int d0, int width,
                                                 float scale, bool wide) {
  for (int e = threadIdx.x; e < kChunkTokens * (kDepth / 4); e += kTileThreads) {
    const int t = e % kChunkTokens, d = (e / kChunkTokens) * 4;
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (t < n) {
      const T* p = src + (size_t)t * stride + d0 + d;
      if (wide && d0 + d < width) ld4(p, x);
      else if (!wide) {
#pragma unroll
        for (int u = 0; u < 4; ++u) if (d0 + d + u < width) x[u] = to_f32(p[u]);
      }
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) dst[d + u][t] = x[u] * scale;
  }
}

// acc[i][j] += sum over `depth` of A[d][4 ty + i] * B[d][4 tx + j]
__device__ __forceinline__ void tile_product(float (&acc)[4][4], const float (*A)[kPad], const float (*B)[kPad], int depth, int ty, int tx) {
#pragma unroll 8
  for (int d = 0; d < depth; ++d) {
    float x[4], y[4];
    ld4(&A[d][ty * 4], x);
    ld4(&B[d][tx * 4], y);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
  }
}

// grid (chunks, heads, tiles of dk x tiles of dv + 1): block z is a tile of what the chunk adds to the state, the last block
// the chunk's score matrix.
template <typename T>
__global__ void __launch_bounds__(kTileThreads) memory_chunk_kernel(MemoryArgs a) {
  __shared__ __align__(16) float As[kChunkTokens][kPad];
  __shared__ __align__(16) float Bs[kChunkTokens][kPad];
  __shared__ double sF[kChunkTokens];
  __shared__ float sI[kChunkTokens], sW[kChunkTokens];
  __shared__ double carry;
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, t0 = it.y, n = it.z - it.y;
  const int tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const int nv = (a.dv + kCols - 1) / kCols, nk = (a.dk + kCols - 1) / kCols;
  const size_t cell = (size_t)it.w * a.heads + head;
  const T* kg = (const T*)a.k + (size_t)t0 * a.k_stride + (size_t)head * a.dk;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  chunk_gates<T>(a, t0, n, head, sF, sI, &carry);
  const bool wide_k = a.dk % 4 == 0 && a.k_stride % 4 == 0 && (uintptr_t)a.k % (4 * sizeof(T)) == 0;

  if ((int)blockIdx.z < nk * nv) {
    const int d0 = (blockIdx.z / nv) * kCols, c0 = (blockIdx.z % nv) * kCols;
    // weights of the tokens at the chunk's end, scaled by the largest of them
    if (tid < 32) {
      const float w0 = (float)(sF[n - 1] - sF[tid]) + sI[tid], w1 = (float)(sF[n - 1] - sF[tid + 32]) + sI[tid + 32];
      const float top = warp_max(fmaxf(w0, w1));
      sW[tid] = tid < n ? expf(w0 - top) : 0.f;
      sW[tid + 32] = tid + 32 < n ? expf(w1 - top) : 0.f;
      if (tid == 0 && blockIdx.z == 0) { a.ends[2 * cell] = (float)sF[n - 1]; a.ends[2 * cell + 1] = top; }
    }
    __syncthreads();
    const T* vg = (const T*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv;
    const bool wide_v = a.dv % 4 == 0 && a.v_stride % 4 == 0 && (uintptr_t)a.v % (4 * sizeof(T)) == 0;
    for (int e = tid; e < kChunkTokens * (kCols / 4); e += kTileThreads) {
      const int t = e / (kCols / 4), c = (e % (kCols / 4)) * 4;
      float kk[4] = {0.f, 0.f, 0.f, 0.f}, vv[4] = {0.f, 0.f, 0.f, 0.f};
      if (t < n) {
        const T* kp = kg + (size_t)t * a.k_stride + d0 + c;
        const T* vp = vg + (size_t)t * a.v_stride + c0 + c;
        if (wide_k) { if (d0 + c < a.dk) ld4(kp, kk); }
        else {
#pragma unroll
          for (int u = 0; u < 4; ++u) if (d0 + c + u < a.dk) kk[u] = to_f32(kp[u]);
        }
        if (wide_v) { if (c0 + c < a.dv) ld4(vp, vv); }
        else {
#pragma unroll
          for (int u = 0; u < 4; ++u) if (c0 + c + u < a.dv) vv[u] = to_f32(vp[u]);
        }
        const float w = sW[t];
#pragma unroll
        for (int u = 0; u < 4; ++u) kk[u] *= w;
      }
      st4(&As[t][c], kk);
      st4(&Bs[t][c], vv);
    }
    __syncthreads();
    tile_product(acc, As, Bs, n, ty, tx);
    float* dst = a.added + cell * ((size_t)a.dk * a.dv + a.dk);
    const bool wide_out = a.dv % 4 == 0 && a.dk % 4 == 0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = d0 + ty * 4 + i, c = c0 + tx * 4;
      if (r >= a.dk) continue;
      if (wide_out) { if (c < a.dv) st4(dst + (size_t)r * a.dv + c, acc[i]); }
      else {
#pragma unroll
        for (int j = 0; j < 4; ++j) if (c + j < a.dv) dst[(size_t)r * a.dv + c + j] = acc[i][j];
      }
    }
    if (c0 == 0 && tid < kCols && d0 + tid < a.dk) {           // the vector n: the weighted sum of the keys
      float s = 0.f;
      for (int t = 0; t < n; ++t) s += As[t][tid];
      dst[(size_t)a.dk * a.dv + d0 + tid] = s;
    }
    return;
  }

  // the score matrix: acc[i][j] = q of token 4 ty + i . k of token 4 tx + j
  const T* qg = (const T*)a.q + (size_t)t0 * a.q_stride + (size_t)head * a.dk;
  const bool wide_q = a.dk % 4 == 0 && a.q_stride % 4 == 0 && (uintptr_t)a.q % (4 * sizeof(T)) == 0;
  for (int d0 = 0; d0 < a.dk; d0 += kDepth) {
    __syncthreads();
    stage_transposed<T>(As, qg, a.q_stride, n, d0, a.dk, a.q_scale, wide_q);
    stage_transposed<T>(Bs, kg, a.k_stride, n, d0, a.dk, 1.0f, wide_k);
    __syncthreads();
    tile_product(acc, As, Bs, kDepth, ty, tx);
  }
  // gates: token s weighs exp(F_t - F_s + i_s - top_t) in the output of token t >= s, top_t the largest exponent of the row
  float* scores = a.scores + cell * (kChunkTokens * kChunkTokens);
  float* rows = a.rows + cell * (3 * kChunkTokens);
  float p[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i;
    float x[4], top = -INFINITY;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = tx * 4 + j;
      x[j] = (s <= t && s < n) ? (float)(sF[t] - sF[s]) + sI[s] : -INFINITY;
      top = fmaxf(top, x[j]);
    }
#pragma unroll
    for (int off = 8; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));   // the 16 threads of a row
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      p[j][i] = x[j] == -INFINITY ? 0.f : expf(x[j] - top) * acc[i][j];
      sum += p[j][i];
    }
#pragma unroll
    for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
    if (tx == 0) {
      rows[t] = (float)sF[t];
      rows[kChunkTokens + t] = top;
      rows[2 * kChunkTokens + t] = sum;
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) st4(scores + (size_t)(tx * 4 + j) * kChunkTokens + ty * 4, p[j]);
}

// spans: (request, first chunk item, end chunk item, -) per long portion.  Walks the chunks in order: `added` of a chunk
// becomes the state BEFORE it, the state after the last chunk goes to the slot (m is left to the output kernel, which runs
// after every block of this one has read the slot's).
__global__ void __launch_bounds__(256) memory_prefix_kernel(MemoryArgs a, const int4* __restrict__ spans) {
  const int4 sp = spans[blockIdx.x];
  const int head = blockIdx.y;
  const long long per = (long long)a.dk * a.dv + a.dk;
  const int tiles = (a.dv + kCols - 1) / kCols;
  float* slot = a.state + (size_t)a.state_slot[sp.x] * a.slot_stride;
  const float m0 = slot[m_offset(a, 0) + head];
  for (long long e = (long long)blockIdx.z * blockDim.x + threadIdx.x; e < per; e += (long long)gridDim.z * blockDim.x) {
    const bool is_n = e >= (long long)a.dk * a.dv;
    float* home = is_n ? slot + n_offset(a, 0) + (size_t)head * a.dk + (e - (long long)a.dk * a.dv)
                       : slot + (size_t)head * a.dk * a.dv + e;
    float S = *home, m = m0;
    for (int c = sp.y; c < sp.z; c += 4) {                    // four chunks' values are asked for together
      const int cnt = min(4, sp.z - c);
      float v[4], F[4], top[4];
      size_t cell[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (u < cnt) {
          cell[u] = (size_t)a.items[c + u].w * a.heads + head;
          v[u] = a.added[cell[u] * per + e];
          F[u] = a.ends[2 * cell[u]];
          top[u] = a.ends[2 * cell[u] + 1];
        }
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        if (u < cnt) {
          a.added[cell[u] * per + e] = S;
          if (e == 0) a.m_before[cell[u]] = m;
          const float m_new = fmaxf(F[u] + m, top[u]);
          S = fmaf(expf(F[u] + m - m_new), S, expf(top[u] - m_new) * v[u]);
          m = m_new;
        }
      }
    }
    *home = S;
    if (is_n)
      for (int t = 1; t < tiles; ++t) home[(size_t)t * a.heads * a.dk] = S;
  }
}

// grid (chunks, heads, tiles of dv).  last_chunk[item] != 0 marks the last chunk of a portion: its blocks leave the running
// maximum in the slot.
template <typename T>
__global__ void __launch_bounds__(kTileThreads) memory_output_kernel(MemoryArgs a, const int* __restrict__ last_chunk) {
  __shared__ __align__(16) float As[kDepth][kPad];
  __shared__ __align__(16) float Bs[kDepth][kPad];
  __shared__ float sN[kDepth];
  __shared__ float s_inter[kChunkTokens], s_intra[kChunkTokens], s_inv[kChunkTokens];
  __shared__ float s_m[kChunkTokens];
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, c0 = blockIdx.z * kCols, t0 = it.y, n = it.z - it.y;
  const int tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const size_t cell = (size_t)it.w * a.heads + head;
  const float* before = a.added + cell * ((size_t)a.dk * a.dv + a.dk);
  const float* n_before = before + (size_t)a.dk * a.dv;
  const float* rows = a.rows + cell * (3 * kChunkTokens);
  if (tid < kChunkTokens) {
    const float from_start = rows[tid] + a.m_before[cell], top = rows[kChunkTokens + tid];
    const float m = fmaxf(from_start, top);
    s_inter[tid] = expf(from_start - m);
    s_intra[tid] = expf(top - m);
    s_m[tid] = m;
  }
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const T* qg = (const T*)a.q + (size_t)t0 * a.q_stride + (size_t)head * a.dk;
  const bool wide_q = a.dk % 4 == 0 && a.q_stride % 4 == 0 && (uintptr_t)a.q % (4 * sizeof(T)) == 0;
  const bool wide_s = a.dv % 4 == 0 && a.dk % 4 == 0;
  float qn = 0.f;                       // thread tid: a quarter of n . q of token tid / 4
  for (int d0 = 0; d0 < a.dk; d0 += kDepth) {
    __syncthreads();
    stage_transposed<T>(As, qg, a.q_stride, n, d0, a.dk, a.q_scale, wide_q);
    for (int e = tid; e < kDepth * (kCols / 4); e += kTileThreads) {
      const int d = e / (kCols / 4), c = (e % (kCols / 4)) * 4;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (d0 + d < a.dk) {
        const float* p = before + (size_t)(d0 + d) * a.dv + c0 + c;
        if (wide_s) { if (c0 + c < a.dv) ld4(p, x); }
        else {
#pragma unroll
          for (int u = 0; u < 4; ++u) if (c0 + c + u < a.dv) x[u] = p[u];
        }
      }
      st4(&Bs[d][c], x);
    }
    if (tid < kDepth) sN[tid] = d0 + tid < a.dk ? n_before[d0 + tid] : 0.f;
    __syncthreads();
    tile_product(acc, As, Bs, kDepth, ty, tx);
    const int t = tid / 4;
#pragma unroll
    for (int d = tid % 4; d < kDepth; d += 4) qn = fmaf(As[d][t], sN[d], qn);
  }
  qn += __shfl_xor_sync(0xffffffffu, qn, 1);
  qn += __shfl_xor_sync(0xffffffffu, qn, 2);
  if (tid % 4 == 0) {
    const int t = tid / 4;
    const float nq = fmaf(s_inter[t], qn, s_intra[t] * rows[2 * kChunkTokens + t]);
    s_inv[t] = 1.0f / (fmaxf(fabsf(nq), expf(-s_m[t])) + a.eps);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float g = s_inter[ty * 4 + i];
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] *= g;
  }
  const float* scores = a.scores + cell * (kChunkTokens * kChunkTokens);
  const T* vg = (const T*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv;
  const bool wide_v = a.dv % 4 == 0 && a.v_stride % 4 == 0 && (uintptr_t)a.v % (4 * sizeof(T)) == 0;
  for (int s0 = 0; s0 < n; s0 += kDepth) {
    __syncthreads();
    for (int e = tid; e < kDepth * (kCols / 4); e += kTileThreads) {
      const int d = e / (kCols / 4), c = (e % (kCols / 4)) * 4, s = s0 + d;
      float x[4], y[4] = {0.f, 0.f, 0.f, 0.f};
      ld4(scores + (size_t)s * kChunkTokens + c, x);
#pragma unroll
      for (int u = 0; u < 4; ++u) x[u] *= s_intra[c + u];
      st4(&As[d][c], x);
      if (s < n) {
        const T* p = vg + (size_t)s * a.v_stride + c0 + c;
        if (wide_v) { if (c0 + c < a.dv) ld4(p, y); }
        else {
#pragma unroll
          for (int u = 0; u < 4; ++u) if (c0 + c + u < a.dv) y[u] = to_f32(p[u]);
        }
      }
      st4(&Bs[d][c], y);
    }
    __syncthreads();
    tile_product(acc, As, Bs, kDepth, ty, tx);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i;
    if (t >= n) continue;
    const float inv = s_inv[t];
    float* o = a.out + (size_t)(t0 + t) * a.out_stride + (size_t)head * a.dv + c0 + tx * 4;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c0 + tx * 4 + j < a.dv) o[j] = acc[i][j] * inv;
  }
  if (last_chunk[blockIdx.x] && tid == 0)
    a.state[(size_t)a.state_slot[it.x] * a.slot_stride + m_offset(a, blockIdx.z) + head] = s_m[n - 1];
}

template <typename T>
static int launch_memory_scan(const MemoryArgs& a, int n_items, cudaStream_t s) {
  const dim3 grid(n_items, a.heads, ceil_div(a.dv, kCols)), block(kWarps * 32);
  const int r = ceil_div(a.dk, kWarps);
  if (r <= 4) return launch_pdl(memory_scan_kernel<T, 4>, grid, block, 0, s, a);
  if (r <= 8) return launch_pdl(memory_scan_kernel<T, 8>, grid, block, 0, s, a);
  if (r <= 16) return launch_pdl(memory_scan_kernel<T, 16>, grid, block, 0, s, a);
  if (r <= 32) return launch_pdl(memory_scan_kernel<T, 32>, grid, block, 0, s, a);
  return launch_pdl(memory_scan_kernel<T, 64>, grid, block, 0, s, a);
}

template <typename T>
static int launch_memory_chunks(const MemoryArgs& a, int n_chunks, const int4* spans, int n_spans, const int* last_chunk, cudaStream_t s) {
  const int nk = ceil_div(a.dk, kCols), nv = ceil_div(a.dv, kCols);
  memory_chunk_kernel<T><<<dim3(n_chunks, a.heads, nk * nv + 1), kTileThreads, 0, s>>>(a);
  const long long per = (long long)a.dk * a.dv + a.dk;
  long long z = (per + 255) / 256;
  if (z > 1024) z = 1024;
  memory_prefix_kernel<<<dim3(n_spans, a.heads, (unsigned)z), 256, 0, s>>>(a, spans);
  memory_output_kernel<T><<<dim3(n_chunks, a.heads, nv), kTileThreads, 0, s>>>(a, last_chunk);
  return LMSF_LAUNCH_STATUS();
}

}  // namespace lmsf

LMSF_API int lmsf_matrix_memory_chunk_tokens() { return lmsf::kChunkTokens; }

// Floats of a state slot, and of the scratch that `n_chunks` chunks of long portions need.
LMSF_API long long lmsf_matrix_memory_state_floats(int heads, int dk, int dv) {
  const long long tiles = (dv + lmsf::kCols - 1) / lmsf::kCols;
  return (long long)heads * dk * (dv + tiles) + tiles * heads;
}
LMSF_API long long lmsf_matrix_memory_scratch_floats(int n_chunks, int heads, int dk, int dv) {
  const long long c = lmsf::kChunkTokens;
  return (long long)n_chunks * heads * ((long long)dk * dv + dk + c * c + 3 * c + 3) + 64;
}

// items (int32 [n_items][4], may be null): (request, first token, end token, chunk index).  n_spans = 0: every item (null: every
// request) token by token.  n_spans > 0: the items are chunks of at most 64 tokens of long portions, `spans` names each
// portion's (request, first item, end item, 0) and last_chunk [n_items] marks the last chunk of each; scratch holds
// lmsf_matrix_memory_scratch_floats(n_items, ...) floats (16-byte aligned).  gi, gf: columns of gate logits (row stride g_stride).
LMSF_API int lmsf_matrix_memory(const void* q, const void* k, const void* v, long long q_stride, long long k_stride,
                                long long v_stride, const void* gi, const void* gf, long long g_stride, const float* bi,
                                const float* bf, float cap, float q_scale, float eps, float* out, long long out_stride,
                                float* state, long long slot_stride, const int* cu_q, const int* state_slot, int n_items,
                                int heads, int dk, int dv, int dtype, const int* items, const int* spans, int n_spans,
                                const int* last_chunk, float* scratch, void* stream) {
  using namespace lmsf;
  if (n_items <= 0) return 0;
  if (heads <= 0 || heads > 65535 || dk <= 0 || dk > kMaxDk || dv <= 0)
    LMSF_REFUSE("matrix_memory: heads=%d dk=%d dv=%d (dk up to %d)", heads, dk, dv, kMaxDk);
  if (ceil_div(dv, kCols) * ceil_div(dk, kCols) + 1 > 65535) LMSF_REFUSE("matrix_memory: dv=%d is too wide", dv);
  if (!(cap > 0.f)) LMSF_REFUSE("matrix_memory: the gates' cap must be positive");
  if (slot_stride < lmsf_matrix_memory_state_floats(heads, dk, dv)) LMSF_REFUSE("matrix_memory: a state slot is too small");
  if (n_spans > 0 && (!items || !spans || !last_chunk || !scratch || (uintptr_t)scratch % 16))
    LMSF_REFUSE("matrix_memory: chunks need their list, their portions and a 16-byte aligned scratch");
  MemoryArgs a{q, k, v, q_stride, k_stride, v_stride, gi, gf, g_stride, bi, bf, cap, q_scale, eps, out, out_stride, state,
               slot_stride, cu_q, state_slot, heads, dk, dv, (const int4*)items, nullptr, nullptr, nullptr, nullptr, nullptr};
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("matrix_memory: unknown dtype code %d", dtype);
  if (n_spans <= 0) return dtype == LMSF_F32 ? launch_memory_scan<float>(a, n_items, s) : launch_memory_scan<bf16>(a, n_items, s);
  const long long cells = (long long)n_items * heads;
  a.scores = scratch;                                         // the parts that are read 16 bytes at a time come first
  a.added = a.scores + cells * kChunkTokens * kChunkTokens;
  a.rows = a.added + (cells * ((long long)dk * dv + dk) + 3) / 4 * 4;
  a.ends = a.rows + cells * 3 * kChunkTokens;
  a.m_before = a.ends + cells * 2;
  return dtype == LMSF_F32 ? launch_memory_chunks<float>(a, n_items, (const int4*)spans, n_spans, last_chunk, s)
                           : launch_memory_chunks<bf16>(a, n_items, (const int4*)spans, n_spans, last_chunk, s);
}
