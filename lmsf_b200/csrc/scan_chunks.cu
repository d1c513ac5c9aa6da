// The plain rule of gated_scan (recurrent.cu) in two other forms, for the same state slots:
//
//   dt = softplus(raw_dt + dt_bias[h]);  a = exp(-exp(a_log[h]) dt);  S <- a S + dt k v^T;  o = S^T q + skip[h] v
//
//   * single tokens (a decode step): one launch that reads and writes the state once, 16 bytes an access, with the token's step
//     size and decay computed where they are used;
//   * long portions: chunks of 64 tokens that run in parallel.  With F the sum of log a since the chunk's start (added up in double,
//     so that differences of large sums stay exact), token s leaves exp(F_end - F_s) dt_s k_s v_s^T in the state at the chunk's end
//     and exp(F_t - F_s) dt_s (k_s . q_t) v_s in the output of token t >= s; every exponent is at most zero:
//       scan_scores_kernel   per chunk and q/k head: the products k_s . q_t (shared by the heads of a group)
//       scan_added_kernel    per chunk and head: what the chunk adds to the state, in tiles
//       scan_prefix_kernel   walks every portion's chunks in order: the state before each chunk; the slot's state afterwards
//       scan_output_kernel   per chunk and head: one product [exp(F_t) q_t | gated scores] x [state before; v], then the skip
//
// q, k and v have the activation type; decays, step sizes, the state and every sum are float32.  float32 activations run on the FMA
// units.  bfloat16 activations run the products of the chunks on the tensor cores (mma.sync) without giving up float32: of the two
// factors of every product one is q, k or v, which IS a bfloat16 number, and the other, a float32 number (a weighted v, the state, a
// gated score), is the sum of three bfloat16 numbers of 8 digits each, which are multiplied one after the other into one float32
// accumulator.  There the scores are made where they are used and scan_scores_kernel falls away.
// A slot holds [head][dv][dk]; the scratch of the chunks holds [dk][dv].
#include "attention_mma.cuh"   // ldmatrix and mma helpers

LMSF_DEFINE_LAST_ERROR(lmsf_scan_chunks)

namespace lmsf {

constexpr int kC = 64;                 // tokens per chunk
constexpr int kThreads = 256;          // 16 x 16 threads, 4 x 4 results each
constexpr int kPad = 68;               // floats of a staged row: 16-byte aligned, neighbouring rows on other banks
constexpr int kDepth = 32;             // inner dimension staged at a time

struct Args {
  float* out; long long out_stride;                 // [n, H * dv]
  const void* q; const void* k; const void* v;      // q, k: [n, G * dk]; v: [n, H * dv]
  long long q_stride, k_stride, v_stride;
  const void* dt; long long dt_stride;              // [n, H] raw step sizes
  const float* dt_bias; const float* a_log; const float* skip;   // [H]
  float* state; long long slot_stride;
  const int* cu_q; const int* state_slot;
  int H, G, dk, dv;
  const int4* items;                                // chunks: (request, first token, end token, chunk number)
  float* scores;                                    // [chunks][G][64 s][64 t]
  float* added;                                     // [chunks][H][dk][dv]: what a chunk adds, then the state before it
  float* ends;                                      // [chunks][H]: the log of the chunk's whole decay
};

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }

// four values of a row from column c on, zeros from `width` on
template <typename T> __device__ __forceinline__ void row4(const T* p, int c, int width, bool wide, float (&x)[4]) {
  x[0] = x[1] = x[2] = x[3] = 0.f;
  if (wide) { if (c < width) ld4(p + c, x); }
  else {
#pragma unroll
    for (int u = 0; u < 4; ++u) if (c + u < width) x[u] = to_f32(p[c + u]);
  }
}
template <typename T> __device__ __forceinline__ bool takes4(const void* p, long long stride, int width) {
  return width % 4 == 0 && stride % 4 == 0 && (uintptr_t)p % (4 * sizeof(T)) == 0;
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
__device__ __forceinline__ void clear(float (&acc)[4][4]) {
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
}

// columns [d0, d0 + kDepth) of a chunk's rows, transposed into dst[column][token], each token times f[token] (null: as it is)
template <typename T>
__device__ __forceinline__ void stage_transposed(float (*dst)[kPad], const T* __restrict__ src, long long stride, int n, int d0, int width,
                                                 const float* f, bool wide) {
  for (int e = threadIdx.x; e < kC * (kDepth / 4); e += kThreads) {
    const int t = e % kC, d = (e / kC) * 4;
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (t < n) row4<T>(src + (size_t)t * stride, d0 + d, width, wide, x);
    const float s = f ? f[t] : 1.f;
#pragma unroll
    for (int u = 0; u < 4; ++u) dst[d + u][t] = x[u] * s;
  }
}

// the chunk's step sizes and summed log decays of a head, by the first 64 threads; every thread of the block calls it
template <typename T>
__device__ __forceinline__ void chunk_steps(const Args& a, int t0, int n, int head, double* sF, float* sDt, double* carry) {
  const int t = threadIdx.x, lane = t & 31;
  double F = 0.0;
  if (t < kC) {
    float dt = 0.f;
    if (t < n) {
      dt = softplus_f(to_f32(((const T*)a.dt)[(size_t)(t0 + t) * a.dt_stride + head]) + a.dt_bias[head]);
      F = (double)(-expf(a.a_log[head]) * dt);
    }
    sDt[t] = dt;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const double p = __shfl_up_sync(0xffffffffu, F, off);
      if (lane >= off) F += p;
    }
    if (t == 31) *carry = F;
  }
  __syncthreads();
  if (t < kC) sF[t] = t >= 32 ? F + *carry : F;
  __syncthreads();
}

// grid (chunks, G)
template <typename T>
__global__ void __launch_bounds__(kThreads) scan_scores_kernel(const Args a) {
  __shared__ __align__(16) float As[kDepth][kPad];
  __shared__ __align__(16) float Bs[kDepth][kPad];
  pdl_launch_dependents();
  pdl_wait();
  const int4 it = a.items[blockIdx.x];
  const int g = blockIdx.y, t0 = it.y, n = it.z - it.y, tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  const T* q = (const T*)a.q + (size_t)t0 * a.q_stride + (size_t)g * a.dk;
  const T* k = (const T*)a.k + (size_t)t0 * a.k_stride + (size_t)g * a.dk;
  const bool wq = takes4<T>(a.q, a.q_stride, a.dk), wk = takes4<T>(a.k, a.k_stride, a.dk);
  float acc[4][4];
  clear(acc);
  for (int d0 = 0; d0 < a.dk; d0 += kDepth) {
    __syncthreads();
    stage_transposed<T>(As, k, a.k_stride, n, d0, a.dk, nullptr, wk);
    stage_transposed<T>(Bs, q, a.q_stride, n, d0, a.dk, nullptr, wq);
    __syncthreads();
    tile_product(acc, As, Bs, min(kDepth, a.dk - d0), ty, tx);
  }
  float* dst = a.scores + ((size_t)it.w * a.G + g) * (kC * kC);
#pragma unroll
  for (int i = 0; i < 4; ++i) st4(dst + (size_t)(ty * 4 + i) * kC + tx * 4, acc[i]);
}

// grid (chunks, H, tiles of dk x tiles of dv)
template <typename T>
__global__ void __launch_bounds__(kThreads) scan_added_kernel(const Args a) {
  __shared__ __align__(16) float As[kC][kPad];        // k: [token][dk]
  __shared__ __align__(16) float Bs[kC][kPad];        // v times its weight: [token][dv]
  __shared__ double sF[kC];
  __shared__ float sDt[kC];
  __shared__ double carry;
  pdl_launch_dependents();
  pdl_wait();
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, t0 = it.y, n = it.z - it.y, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const int nv = (a.dv + 63) / 64, d0 = (blockIdx.z / nv) * 64, c0 = (blockIdx.z % nv) * 64;
  const size_t cell = (size_t)it.w * a.H + head;
  const T* k = (const T*)a.k + (size_t)t0 * a.k_stride + (size_t)(head / (a.H / a.G)) * a.dk;
  const T* v = (const T*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv;
  const bool wk = takes4<T>(a.k, a.k_stride, a.dk), wv = takes4<T>(a.v, a.v_stride, a.dv);
  chunk_steps<T>(a, t0, n, head, sF, sDt, &carry);
  if (tid == 0 && blockIdx.z == 0) a.ends[cell] = (float)sF[n - 1];
  for (int e = tid; e < kC * 16; e += kThreads) {
    const int t = e / 16, c = (e % 16) * 4;
    float x[4] = {0.f, 0.f, 0.f, 0.f}, y[4] = {0.f, 0.f, 0.f, 0.f};
    if (t < n) {
      row4<T>(k + (size_t)t * a.k_stride, d0 + c, a.dk, wk, x);
      row4<T>(v + (size_t)t * a.v_stride, c0 + c, a.dv, wv, y);
      const float w = expf((float)(sF[n - 1] - sF[t])) * sDt[t];
#pragma unroll
      for (int u = 0; u < 4; ++u) y[u] *= w;
    }
    st4(&As[t][c], x);
    st4(&Bs[t][c], y);
  }
  __syncthreads();
  float acc[4][4];
  clear(acc);
  tile_product(acc, As, Bs, n, ty, tx);
  float* dst = a.added + cell * ((size_t)a.dk * a.dv);
  const bool wide = a.dv % 4 == 0;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = d0 + ty * 4 + i, c = c0 + tx * 4;
    if (r >= a.dk) continue;
    if (wide) { if (c < a.dv) st4(dst + (size_t)r * a.dv + c, acc[i]); }
    else {
#pragma unroll
      for (int j = 0; j < 4; ++j) if (c + j < a.dv) dst[(size_t)r * a.dv + c + j] = acc[i][j];
    }
  }
}

// grid (portions, H, parts of dk * dv).  spans: (request, first chunk item, end chunk item, -).  V values of a row a thread.
template <int V>
__global__ void __launch_bounds__(128) scan_prefix_kernel(const Args a, const int4* __restrict__ spans) {
  pdl_launch_dependents();
  pdl_wait();
  const int4 sp = spans[blockIdx.x];
  const int head = blockIdx.y, per = a.dk * a.dv;
  float* slot = a.state + (size_t)a.state_slot[sp.x] * a.slot_stride + (size_t)head * per;
  for (int e = (blockIdx.z * blockDim.x + threadIdx.x) * V; e < per; e += gridDim.z * blockDim.x * V) {
    float* home = slot + (size_t)(e % a.dv) * a.dk + e / a.dv;
    float S[V];
#pragma unroll
    for (int i = 0; i < V; ++i) S[i] = home[(size_t)i * a.dk];
    for (int c = sp.y; c < sp.z; c += 8) {                    // eight chunks' values are asked for together
      const int cnt = min(8, sp.z - c);
      float x[8][V], F[8];
      size_t cell[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (u < cnt) {
          cell[u] = (size_t)a.items[c + u].w * a.H + head;
          const float* p = a.added + cell[u] * per + e;
          if constexpr (V == 4) ld4(p, x[u]); else x[u][0] = *p;
          F[u] = a.ends[cell[u]];
        }
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (u < cnt) {
          float* p = a.added + cell[u] * per + e;
          if constexpr (V == 4) st4(p, S); else *p = S[0];
          const float f = expf(F[u]);
#pragma unroll
          for (int i = 0; i < V; ++i) S[i] = fmaf(f, S[i], x[u][i]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < V; ++i) home[(size_t)i * a.dk] = S[i];
  }
}

// grid (chunks, H, tiles of dv)
template <typename T>
__global__ void __launch_bounds__(kThreads) scan_output_kernel(const Args a) {
  __shared__ __align__(16) float As[kDepth][kPad];     // [dk or token s][token t]
  __shared__ __align__(16) float Bs[kDepth][kPad];     // [dk or token s][dv]
  __shared__ double sF[kC];
  __shared__ float sDt[kC], sE[kC];
  __shared__ double carry;
  pdl_launch_dependents();
  pdl_wait();
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, c0 = blockIdx.z * 64, t0 = it.y, n = it.z - it.y, tid = threadIdx.x, tx = tid % 16, ty = tid / 16;
  const int g = head / (a.H / a.G);
  const T* q = (const T*)a.q + (size_t)t0 * a.q_stride + (size_t)g * a.dk;
  const T* v = (const T*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv;
  const bool wq = takes4<T>(a.q, a.q_stride, a.dk), wv = takes4<T>(a.v, a.v_stride, a.dv);
  const float* before = a.added + ((size_t)it.w * a.H + head) * ((size_t)a.dk * a.dv);
  const float* scores = a.scores + ((size_t)it.w * a.G + g) * (kC * kC);
  chunk_steps<T>(a, t0, n, head, sF, sDt, &carry);
  if (tid < kC) sE[tid] = expf((float)sF[tid]);
  float acc[4][4];
  clear(acc);
  for (int d0 = 0; d0 < a.dk; d0 += kDepth) {
    __syncthreads();
    stage_transposed<T>(As, q, a.q_stride, n, d0, a.dk, sE, wq);
    for (int e = tid; e < kDepth * 16; e += kThreads) {
      const int d = e / 16, c = (e % 16) * 4;
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (d0 + d < a.dk) row4<float>(before + (size_t)(d0 + d) * a.dv, c0 + c, a.dv, a.dv % 4 == 0, x);
      st4(&Bs[d][c], x);
    }
    __syncthreads();
    tile_product(acc, As, Bs, min(kDepth, a.dk - d0), ty, tx);
  }
  for (int s0 = 0; s0 < n; s0 += kDepth) {
    __syncthreads();
    for (int e = tid; e < kDepth * 16; e += kThreads) {
      const int d = e / 16, c = (e % 16) * 4, s = s0 + d;
      float x[4] = {0.f, 0.f, 0.f, 0.f}, y[4] = {0.f, 0.f, 0.f, 0.f};
      if (s < n) {
        ld4(scores + (size_t)s * kC + c, x);
        row4<T>(v + (size_t)s * a.v_stride, c0 + c, a.dv, wv, y);
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) x[u] = (s <= c + u && s < n) ? x[u] * (expf((float)(sF[c + u] - sF[s])) * sDt[s]) : 0.f;
      st4(&As[d][c], x);
      st4(&Bs[d][c], y);
    }
    __syncthreads();
    tile_product(acc, As, Bs, min(kDepth, n - s0), ty, tx);
  }
  const float skip = a.skip ? a.skip[head] : 0.f;
  const bool wide = a.dv % 4 == 0 && a.out_stride % 4 == 0 && (uintptr_t)a.out % 16 == 0;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i, c = c0 + tx * 4;
    if (t >= n) continue;
    float x[4];
    row4<T>(v + (size_t)t * a.v_stride, c, a.dv, wv, x);
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(skip, x[j], acc[i][j]);
    float* o = a.out + (size_t)(t0 + t) * a.out_stride + (size_t)head * a.dv + c;
    if (wide) { if (c < a.dv) st4(o, acc[i]); }
    else {
#pragma unroll
      for (int j = 0; j < 4; ++j) if (c + j < a.dv) o[j] = acc[i][j];
    }
  }
}

// ------------------------------------------------------------------------------------------------ chunks on the tensor cores
using fa::ldmatrix_x4;
using fa::ldmatrix_x4_trans;
using fa::mma_16816;
using fa::smem_u32;

constexpr int kTile = 64;              // columns of dv and rows of the state per stage
constexpr int kRow = kTile + 8;        // bfloat16 values of a staged row of 64: rows fall on different banks for ldmatrix
constexpr int kWideRow = 128 + 8;

// x as a sum of three bfloat16 numbers (24 digits in all)
__device__ __forceinline__ void split3(float x, bf16 (&s)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) { s[i] = __float2bfloat16_rn(x); x -= __bfloat162float(s[i]); }
}
__device__ __forceinline__ void split3x4(const float (&x)[4], uint2 (&w)[3]) {
  bf16 s[4][3];
#pragma unroll
  for (int u = 0; u < 4; ++u) split3(x[u], s[u]);
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const __nv_bfloat162 lo(s[0][i], s[1][i]), hi(s[2][i], s[3][i]);
    w[i].x = *reinterpret_cast<const uint32_t*>(&lo);
    w[i].y = *reinterpret_cast<const uint32_t*>(&hi);
  }
}

// `cols` columns (a multiple of 8) from c0 on of a chunk's rows into dst [64][ld]; zeros beyond n rows and `width` columns.  Where the
// rows allow it the copies are asynchronous: the caller waits for them (cp_async_wait and a barrier).
template <int NT>
__device__ __forceinline__ void stage_rows(bf16* dst, int ld, const bf16* __restrict__ src, long long stride, int n, int c0, int cols, int width) {
  const bool wide = width % 8 == 0 && stride % 8 == 0 && (uintptr_t)src % 16 == 0;
  const int per_row = cols / 8;
  for (int e = threadIdx.x; e < kC * per_row; e += NT) {
    const int t = e / per_row, c = (e % per_row) * 8;
    const bf16* p = src + (size_t)t * stride + c0 + c;
    if (wide) {
      const bool ok = t < n && c0 + c < width;
      fa::cp_async_16(smem_u32(dst + (size_t)t * ld + c), ok ? p : src, ok ? 16 : 0);
      continue;
    }
    uint4 x = make_uint4(0u, 0u, 0u, 0u);
    bf16* b = reinterpret_cast<bf16*>(&x);
#pragma unroll
    for (int u = 0; u < 8; ++u) if (t < n && c0 + c + u < width) b[u] = p[u];
    *reinterpret_cast<uint4*>(dst + (size_t)t * ld + c) = x;
  }
  fa::cp_async_commit();
}

// grid (chunks, H, tiles of 128 of dk x tiles of 64 of dv); 8 warps, 32 x 32 results each
__global__ void __launch_bounds__(256) scan_added_tc_kernel(const Args a) {
  __shared__ __align__(16) bf16 sK[kC * kWideRow];
  __shared__ __align__(16) bf16 sV[3][kC * kRow];      // v times its weight, in three parts
  __shared__ double sF[kC];
  __shared__ float sDt[kC];
  __shared__ double carry;
  pdl_launch_dependents();
  pdl_wait();
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, t0 = it.y, n = it.z - it.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nv = (a.dv + kTile - 1) / kTile, d0 = (blockIdx.z / nv) * 128, c0 = (blockIdx.z % nv) * kTile;
  const size_t cell = (size_t)it.w * a.H + head;
  const bf16* k = (const bf16*)a.k + (size_t)t0 * a.k_stride + (size_t)(head / (a.H / a.G)) * a.dk;
  const bf16* v = (const bf16*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv;
  const bool wv = takes4<bf16>(a.v, a.v_stride, a.dv);
  // everything that is read from memory is asked for before anything waits
  stage_rows<256>(sK, kWideRow, k, a.k_stride, n, d0, 128, a.dk);
  const int c = (tid % 16) * 4;
  float y[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = tid / 16 + 16 * i;
    y[i][0] = y[i][1] = y[i][2] = y[i][3] = 0.f;
    if (t < n) row4<bf16>(v + (size_t)t * a.v_stride, c0 + c, a.dv, wv, y[i]);
  }
  chunk_steps<bf16>(a, t0, n, head, sF, sDt, &carry);
  if (tid == 0 && blockIdx.z == 0) a.ends[cell] = (float)sF[n - 1];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = tid / 16 + 16 * i;
    const float w = t < n ? expf((float)(sF[n - 1] - sF[t])) * sDt[t] : 0.f;
#pragma unroll
    for (int u = 0; u < 4; ++u) y[i][u] *= w;
    uint2 s[3];
    split3x4(y[i], s);
#pragma unroll
    for (int j = 0; j < 3; ++j) *reinterpret_cast<uint2*>(&sV[j][t * kRow + c]) = s[j];
  }
  fa::cp_async_wait<0>();
  __syncthreads();
  const int m0 = (warp & 3) * 32, n0 = (warp >> 2) * 32, mi = lane >> 3, r = lane & 7, g4 = lane >> 2, t4 = lane & 3;
  float acc[2][4][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f;
#pragma unroll
  for (int ks = 0; ks < kC / 16; ++ks) {
    if (ks * 16 >= n) break;
    uint32_t A[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) ldmatrix_x4_trans(A[i], smem_u32(&sK[(ks * 16 + (mi >> 1) * 8 + r) * kWideRow + m0 + i * 16 + (mi & 1) * 8]));
#pragma unroll
    for (int s = 0; s < 3; ++s)
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        uint32_t B[4];
        ldmatrix_x4_trans(B, smem_u32(&sV[s][(ks * 16 + (mi & 1) * 8 + r) * kRow + n0 + j * 16 + (mi >> 1) * 8]));
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_16816(acc[i][2 * j], A[i], B[0], B[1]);
          mma_16816(acc[i][2 * j + 1], A[i], B[2], B[3]);
        }
      }
  }
  float* dst = a.added + cell * ((size_t)a.dk * a.dv);
  const bool pairs = a.dv % 2 == 0;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int row = d0 + m0 + i * 16 + g4 + h * 8;
      if (row >= a.dk) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int c = c0 + n0 + j * 8 + t4 * 2;
        float* p = dst + (size_t)row * a.dv + c;
        if (pairs) { if (c < a.dv) *reinterpret_cast<float2*>(p) = make_float2(acc[i][j][2 * h], acc[i][j][2 * h + 1]); }
        else {
          if (c < a.dv) p[0] = acc[i][j][2 * h];
          if (c + 1 < a.dv) p[1] = acc[i][j][2 * h + 1];
        }
      }
    }
}

// grid (chunks, H, tiles of 64 of dv); 4 warps, 16 tokens x 64 values each.  Shared memory: q and k [64][dk rounded up to 64, + 8],
// v [64][72], a slice of 64 rows of the state in three parts.
__global__ void __launch_bounds__(128) scan_output_tc_kernel(const Args a) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ double sF[kC];
  __shared__ float sDt[kC];
  __shared__ double carry;
  const int dkp = (a.dk + kTile - 1) / kTile * kTile, ldq = dkp + 8;
  bf16* sQ = reinterpret_cast<bf16*>(smem);
  bf16* sK = sQ + kC * ldq;
  bf16* sV = sK + kC * ldq;
  bf16* sS = sV + kC * kRow;
  pdl_launch_dependents();
  pdl_wait();
  const int4 it = a.items[blockIdx.x];
  const int head = blockIdx.y, c0 = blockIdx.z * kTile, t0 = it.y, n = it.z - it.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = head / (a.H / a.G);
  const float* before = a.added + ((size_t)it.w * a.H + head) * ((size_t)a.dk * a.dv);
  stage_rows<128>(sQ, ldq, (const bf16*)a.q + (size_t)t0 * a.q_stride + (size_t)g * a.dk, a.q_stride, n, 0, dkp, a.dk);
  stage_rows<128>(sK, ldq, (const bf16*)a.k + (size_t)t0 * a.k_stride + (size_t)g * a.dk, a.k_stride, n, 0, dkp, a.dk);
  stage_rows<128>(sV, kRow, (const bf16*)a.v + (size_t)t0 * a.v_stride + (size_t)head * a.dv, a.v_stride, n, c0, kTile, a.dv);
  // a slice of 64 rows of the state on its way in registers: asked for one slice ahead
  const int sc = (tid % 16) * 4;
  float S[8][4];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int d = d0 + tid / 16 + 8 * i;
      S[i][0] = S[i][1] = S[i][2] = S[i][3] = 0.f;
      if (d < a.dk) row4<float>(before + (size_t)d * a.dv, c0 + sc, a.dv, a.dv % 4 == 0, S[i]);
    }
  };
  fetch(0);
  chunk_steps<bf16>(a, t0, n, head, sF, sDt, &carry);
  fa::cp_async_wait<0>();
  const int mi = lane >> 3, r = lane & 7, g4 = lane >> 2, t4 = lane & 3, row0 = warp * 16;
  auto q_frag = [&](uint32_t (&A)[4], int col) { ldmatrix_x4(A, smem_u32(&sQ[(row0 + (mi & 1) * 8 + r) * ldq + col + (mi >> 1) * 8])); };
  float o[8][4];
#pragma unroll
  for (int j = 0; j < 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // what the state before the chunk gives: q times S, the decay since the chunk's start afterwards
  for (int d0 = 0; d0 < dkp; d0 += kTile) {
    if (d0 > 0) __syncthreads();
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      uint2 s[3];
      split3x4(S[i], s);
#pragma unroll
      for (int j = 0; j < 3; ++j) *reinterpret_cast<uint2*>(&sS[(j * kTile + tid / 16 + 8 * i) * kRow + sc]) = s[j];
    }
    __syncthreads();                                              // (the first one also covers q, k and v)
    if (d0 + kTile < dkp) fetch(d0 + kTile);
#pragma unroll
    for (int ks = 0; ks < kTile / 16; ++ks) {
      uint32_t A[4];
      q_frag(A, d0 + ks * 16);
#pragma unroll
      for (int s = 0; s < 3; ++s)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t B[4];
          ldmatrix_x4_trans(B, smem_u32(&sS[(s * kTile + ks * 16 + (mi & 1) * 8 + r) * kRow + j * 16 + (mi >> 1) * 8]));
          mma_16816(o[2 * j], A, B[0], B[1]);
          mma_16816(o[2 * j + 1], A, B[2], B[3]);
        }
    }
  }
  const double F[2] = {sF[row0 + g4], sF[row0 + g4 + 8]};
  const float E[2] = {expf((float)F[0]), expf((float)F[1])};
#pragma unroll
  for (int j = 0; j < 8; ++j) { o[j][0] *= E[0]; o[j][1] *= E[0]; o[j][2] *= E[1]; o[j][3] *= E[1]; }
  // what the chunk's own tokens give, 16 of them at a time up to the warp's own
#pragma unroll
  for (int kb = 0; kb < kC / 16; ++kb) {
    if (kb > warp || kb * 16 >= n) break;
    float p[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    for (int ks = 0; ks < dkp / 16; ++ks) {
      uint32_t A[4], B[4];
      q_frag(A, ks * 16);
      ldmatrix_x4(B, smem_u32(&sK[(kb * 16 + (mi >> 1) * 8 + r) * ldq + ks * 16 + (mi & 1) * 8]));
      mma_16816(p[0], A, B[0], B[1]);
      mma_16816(p[1], A, B[2], B[3]);
    }
    uint32_t P[3][4];
    bf16 part[2][4][3];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int t = row0 + g4 + (e >> 1) * 8, s = kb * 16 + j * 8 + t4 * 2 + (e & 1);
        const float w = (s <= t && s < n) ? expf((float)(F[e >> 1] - sF[s])) * sDt[s] : 0.f;
        split3(p[j][e] * w, part[j][e]);
      }
#pragma unroll
    for (int s = 0; s < 3; ++s)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 x(part[i >> 1][(i & 1) * 2][s], part[i >> 1][(i & 1) * 2 + 1][s]);
        P[s][i] = *reinterpret_cast<const uint32_t*>(&x);
      }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t B[4];
      ldmatrix_x4_trans(B, smem_u32(&sV[(kb * 16 + (mi & 1) * 8 + r) * kRow + j * 16 + (mi >> 1) * 8]));
#pragma unroll
      for (int s = 0; s < 3; ++s) {
        mma_16816(o[2 * j], P[s], B[0], B[1]);
        mma_16816(o[2 * j + 1], P[s], B[2], B[3]);
      }
    }
  }
  const float skip = a.skip ? a.skip[head] : 0.f;
  const bool pairs = a.dv % 2 == 0 && a.out_stride % 2 == 0 && (uintptr_t)a.out % 8 == 0;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int t = row0 + g4 + h * 8;
    if (t >= n) continue;
    float* dst = a.out + (size_t)(t0 + t) * a.out_stride + (size_t)head * a.dv + c0;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int c = j * 8 + t4 * 2;
      const float y0 = fmaf(skip, __bfloat162float(sV[t * kRow + c]), o[j][2 * h]);
      const float y1 = fmaf(skip, __bfloat162float(sV[t * kRow + c + 1]), o[j][2 * h + 1]);
      if (pairs) { if (c0 + c < a.dv) *reinterpret_cast<float2*>(dst + c) = make_float2(y0, y1); }
      else {
        if (c0 + c < a.dv) dst[c] = y0;
        if (c0 + c + 1 < a.dv) dst[c + 1] = y1;
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ single tokens
// grid (tiles of dv, H, requests); 256 threads: eight lanes share a column of the state (its dk values, four at a time, the
// lanes' words side by side), a thread has COLS columns, 32 apart.  VEC: 16-byte accesses of state, q and k.
constexpr int kStepLanes = 8;
template <typename T, int COLS, bool VEC>
__global__ void __launch_bounds__(kThreads) scan_step_kernel(const Args a) {
  __shared__ __align__(16) float sk[256], sq[256];
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y, tid = threadIdx.x, r = tid % kStepLanes;
  const int t = a.cu_q[seq];
  if (a.cu_q[seq + 1] <= t) return;
  const int g = head / (a.H / a.G), dk = a.dk, dv = a.dv;
  const float dt = softplus_f(to_f32(((const T*)a.dt)[(size_t)t * a.dt_stride + head]) + a.dt_bias[head]);
  const float dec = expf(-expf(a.a_log[head]) * dt);
  if (tid < dk) {
    sk[tid] = to_f32(((const T*)a.k)[(size_t)t * a.k_stride + (size_t)g * dk + tid]);
    sq[tid] = to_f32(((const T*)a.q)[(size_t)t * a.q_stride + (size_t)g * dk + tid]);
  }
  __syncthreads();
  float* st = a.state + (size_t)a.state_slot[seq] * a.slot_stride + (size_t)head * dv * dk;
  const int col0 = blockIdx.x * (kThreads / kStepLanes * COLS) + tid / kStepLanes;
  const float skip = a.skip ? a.skip[head] : 0.f;
  float x[COLS], u[COLS], o[COLS];
#pragma unroll
  for (int c = 0; c < COLS; ++c) {
    const int col = col0 + c * (kThreads / kStepLanes);
    x[c] = col < dv ? to_f32(((const T*)a.v)[(size_t)t * a.v_stride + (size_t)head * dv + col]) : 0.f;
    u[c] = dt * x[c];
    o[c] = 0.f;
  }
  if (VEC) {
    for (int i0 = r * 4; i0 < dk; i0 += 4 * kStepLanes) {
      float S[COLS][4], kk[4], qq[4];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const int col = col0 + c * (kThreads / kStepLanes);
        if (col < dv) ld4(st + (size_t)col * dk + i0, S[c]);
      }
      ld4(sk + i0, kk);
      ld4(sq + i0, qq);
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const int col = col0 + c * (kThreads / kStepLanes);
        if (col >= dv) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          S[c][e] = fmaf(kk[e], u[c], dec * S[c][e]);
          o[c] = fmaf(S[c][e], qq[e], o[c]);
        }
        st4(st + (size_t)col * dk + i0, S[c]);
      }
    }
  } else {
    for (int i = r; i < dk; i += kStepLanes) {
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const int col = col0 + c * (kThreads / kStepLanes);
        if (col >= dv) continue;
        const float S = fmaf(sk[i], u[c], dec * st[(size_t)col * dk + i]);
        o[c] = fmaf(S, sq[i], o[c]);
        st[(size_t)col * dk + i] = S;
      }
    }
  }
#pragma unroll
  for (int c = 0; c < COLS; ++c) {
#pragma unroll
    for (int off = kStepLanes / 2; off > 0; off >>= 1) o[c] += __shfl_xor_sync(0xffffffffu, o[c], off);
    const int col = col0 + c * (kThreads / kStepLanes);
    if (r == 0 && col < dv) a.out[(size_t)t * a.out_stride + (size_t)head * dv + col] = fmaf(skip, x[c], o[c]);
  }
}

template <typename T>
static int run_chunks(const Args& a, int n_chunks, const int4* spans, int n_spans, cudaStream_t s) {
  const int nk = ceil_div(a.dk, 64), nv = ceil_div(a.dv, 64);
  constexpr bool kTc = sizeof(T) == 2;
  int rc;
  if constexpr (kTc) {
    rc = launch_pdl(scan_added_tc_kernel, dim3(n_chunks, a.H, ceil_div(a.dk, 128) * nv), dim3(256), 0, s, a);
  } else {
    rc = launch_pdl(scan_scores_kernel<T>, dim3(n_chunks, a.G), dim3(kThreads), 0, s, a);
    if (!rc) rc = launch_pdl(scan_added_kernel<T>, dim3(n_chunks, a.H, nk * nv), dim3(kThreads), 0, s, a);
  }
  const int v4 = a.dv % 4 == 0 ? 4 : 1;
  int parts = ceil_div(a.dk * a.dv, 128 * v4);
  if (parts > 64) parts = 64;
  if (!rc) rc = v4 == 4 ? launch_pdl(scan_prefix_kernel<4>, dim3(n_spans, a.H, parts), dim3(128), 0, s, a, spans)
                        : launch_pdl(scan_prefix_kernel<1>, dim3(n_spans, a.H, parts), dim3(128), 0, s, a, spans);
  if (rc) return rc;
  if constexpr (!kTc) return launch_pdl(scan_output_kernel<T>, dim3(n_chunks, a.H, nv), dim3(kThreads), 0, s, a);
  const int smem = (2 * kC * (ceil_div(a.dk, kTile) * kTile + 8) + 4 * kC * kRow) * (int)sizeof(bf16);
  static int allowed = 0;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(scan_output_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  return launch_pdl(scan_output_tc_kernel, dim3(n_chunks, a.H, nv), dim3(128), smem, s, a);
}

template <typename T>
static int run_step(const Args& a, int n_seqs, cudaStream_t s) {
  const bool vec = a.dk % 4 == 0 && a.slot_stride % 4 == 0 && (uintptr_t)a.state % 16 == 0;
  const int per = kThreads / kStepLanes;               // columns that a block of one column a thread serves
  // as many columns a thread as still leave every SM several blocks
  const long long pairs = (long long)a.H * n_seqs;
  const int cols = (a.dv > 2 * per && pairs >= 592) ? 4 : (a.dv > per && pairs >= 296) ? 2 : 1;
#define LMSF_GO(C) do { dim3 grid(ceil_div(a.dv, per * C), a.H, n_seqs);                                                       \
    return vec ? launch_pdl(scan_step_kernel<T, C, true>, grid, dim3(kThreads), 0, s, a)                                       \
               : launch_pdl(scan_step_kernel<T, C, false>, grid, dim3(kThreads), 0, s, a); } while (0)
  if (cols == 4) LMSF_GO(4);
  if (cols == 2) LMSF_GO(2);
  LMSF_GO(1);
#undef LMSF_GO
}

}  // namespace lmsf

LMSF_API int lmsf_scan_chunk_tokens() { return lmsf::kC; }

// Floats of scratch for n_chunks chunks.
LMSF_API long long lmsf_scan_chunks_scratch_floats(int n_chunks, int H, int G, int dk, int dv) {
  return (long long)n_chunks * ((long long)G * lmsf::kC * lmsf::kC + (long long)H * dk * dv + (H + 3) / 4 * 4);
}

// items [n_chunks] and spans [n_spans] as above (int4 on the device).  n_chunks 0: every request brings one token, n_seqs of them
// (items, spans and scratch are not read).
LMSF_API int lmsf_scan_chunks(float* out, long long out_stride, const void* q, const void* k, const void* v, long long q_stride,
                              long long k_stride, long long v_stride, const void* dt, long long dt_stride, const float* dt_bias,
                              const float* a_log, const float* skip, float* state, long long slot_stride, const int* cu_q,
                              const int* state_slot, int n_seqs, int H, int G, int dk, int dv, const void* items, int n_chunks,
                              const void* spans, int n_spans, float* scratch, int dtype, void* stream) {
  using namespace lmsf;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > 256 || dv <= 0 || H > 65535 || n_seqs > 65535)
    LMSF_REFUSE("scan_chunks: %d heads over %d q/k heads, dk=%d (up to 256), dv=%d", H, G, dk, dv);
  if (dtype != LMSF_F32 && dtype != LMSF_BF16) LMSF_REFUSE("scan_chunks: unknown dtype code %d", dtype);
  Args a{out, out_stride, q, k, v, q_stride, k_stride, v_stride, dt, dt_stride, dt_bias, a_log, skip, state, slot_stride, cu_q,
         state_slot, H, G, dk, dv, (const int4*)items, nullptr, nullptr, nullptr};
  cudaStream_t s = (cudaStream_t)stream;
  if (n_chunks == 0) {
    if (n_seqs <= 0) return 0;
    return dtype == LMSF_F32 ? run_step<float>(a, n_seqs, s) : run_step<bf16>(a, n_seqs, s);
  }
  if (!items || !spans || n_spans <= 0 || !scratch || (uintptr_t)scratch % 16) LMSF_REFUSE("scan_chunks: chunks, portions and a 16-byte aligned scratch are needed");
  a.scores = scratch;
  a.added = a.scores + (size_t)n_chunks * G * kC * kC;
  a.ends = a.added + (size_t)n_chunks * H * dk * dv;
  return dtype == LMSF_F32 ? run_chunks<float>(a, n_chunks, (const int4*)spans, n_spans, s)
                           : run_chunks<bf16>(a, n_chunks, (const int4*)spans, n_spans, s);
}
