// Building blocks of the bfloat16 tensor-core attention kernels: asynchronous copies of key/value
// rows from cache pages into shared memory, ldmatrix fragment loads and the m16n8k16 product.
#pragma once
#include "common.cuh"

namespace lmsf {
namespace fa {

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// 16-byte asynchronous copy; src_bytes = 0 writes zeros and reads nothing.
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, int src_bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(src_bytes));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

// c (16x8, float32) += a (16x16 bf16, row) * b (16x8 bf16, col)
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

constexpr int kTileKeys = 64;   // keys per pipeline stage (prefill; decode blocks may take narrower tiles)
constexpr int kThreads = 128;   // 4 warps

// Geometry of one layer's cache and of one request's block table.  block_size is a power of two.
struct PagedKV {
  const bf16* cache;        // [page][planes][kv_head][slot][HD]
  long long page_stride;    // elements between pages
  int block_size, block_shift;
  int n_kv_heads;
  long long v_off;          // elements from a key's row to its value's row; 0 when one cached vector is both (planes = 1)
};

__host__ inline bool make_paged_kv(PagedKV& kv, const void* cache, long long page_stride, int block_size, int n_kv_heads,
                                   int head_dim, int planes = 2) {
  if (block_size <= 0 || (block_size & (block_size - 1)) || (planes != 1 && planes != 2)) return false;
  int sh = 0;
  while ((1 << sh) < block_size) ++sh;
  kv = PagedKV{(const bf16*)cache, page_stride, block_size, sh, n_kv_heads,
               planes == 2 ? (long long)n_kv_heads * block_size * head_dim : 0};
  return true;
}

// What a design may add to the plain causal softmax of the tensor-core kernels; everything is off when zero or null.
struct ScoreExtras {
  int chunk;            // > 0: a query at position p sees the keys p - p % chunk .. p only (chunks count from position 0)
  const float* r1;      // [n_q_heads] with r2: r1 * ln(1 + r2 * (p - key)) is taken off the scaled score
  const float* r2;
  const float* sinks;   // [n_q_heads]: exp(sink) is one more term of the softmax's denominator, without a key or a value
  int keep_first;       // > 0 (with a window): the request's first keep_first keys stay visible behind the window
  int sigmoid;          // 1: a visible key's weight is sigmoid(score), not normalised over the keys (no softmax, no sinks)
  const float* head_bias;   // [n_q_heads]: a number per query head added to every scaled score
  const float* dist;        // [n_q_heads][dist_n]: the entry of the distance p - key (the last entry for every distance from
  int dist_n;               // dist_n - 1 on) is added to the scaled score
  float softcap;            // > 0: a scaled score s becomes softcap * tanh(s / softcap) before anything else is done to it
};
// tanh(x) / x as a polynomial in u = x^2, of two reaches:
//   |x| <= kTanhNear: the series of tanh at 0 through x^9, within 1e-8 of the quotient
//   |x| <= kTanhFar:  the polynomial of degree 9 in u that meets the quotient at the ten Chebyshev points of [0, kTanhFar^2],
//                     within 2e-8 of it (2e-7 with float32's own rounding)
// and beyond that 1 - 2 / (1 + e^(2x)) on the special-function unit.
constexpr float kTanhNear = 0.25f, kTanhFar = 1.5f;
constexpr float kTanh3 = -1.0f / 3.0f, kTanh5 = 2.0f / 15.0f, kTanh7 = -17.0f / 315.0f, kTanh9 = 62.0f / 2835.0f;
constexpr int kTanhTerms = 10;
__host__ __device__ constexpr float tanh_far_coef(int i) {
  constexpr float c[kTanhTerms] = {0.99999998147f, -0.33333167893f, 0.13330850832f, -0.053820780479f, 0.021412750936f,
                                   -0.0080194525170f, 0.0025848281494f, -6.3165987782e-4f, 9.8872513344e-5f, -7.2078166865e-6f};
  return c[i];
}
constexpr float kTwoLog2e = 2.8853900817779268f;
__device__ __forceinline__ float tanh_score(float x) {
  const float u = x * x;
  float p = tanh_far_coef(kTanhTerms - 1);
#pragma unroll
  for (int i = kTanhTerms - 2; i >= 0; --i) p = fmaf(u, p, tanh_far_coef(i));
  float t = x * p;
  if (fabsf(x) > kTanhFar) {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * kTwoLog2e));
    t = 1.0f - __fdividef(2.0f, 1.0f + e);
  }
  return t;
}
// The key tiles that a block walks when the window's keys [lo, hi) are joined by the kept first keys [0, keep): tiles
// 0 .. n_first - 1 and then tile_lo .. tile_hi - 1 (n_first = 0 when the window's first tile reaches the kept keys anyway).
struct TileRange {
  int n_first, tile_lo, n;
  __device__ __forceinline__ int at(int i) const { return i < n_first ? i : tile_lo + (i - n_first); }
};
__device__ __forceinline__ TileRange tile_range(int lo, int hi, int keep_first, int tile) {
  TileRange r;
  r.tile_lo = lo / tile;
  r.n_first = keep_first > 0 ? min((keep_first + tile - 1) / tile, r.tile_lo) : 0;
  r.n = r.n_first + max(0, (hi + tile - 1) / tile - r.tile_lo);
  return r;
}
// sigmoid of a score given in base-2 units (x * log2(e)): 1 / (1 + 2^-v) from the special-function unit's 2^x and 1/x (each
// within two units of the last place; the weight is rounded to bfloat16 next); -inf gives 0
__device__ __forceinline__ float sigmoid2(float v) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(-v));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + e));
  return r;
}
// what a table of distances adds to a score, in base-2 units; `row` is the head's row of the table
__device__ __forceinline__ float table_bias2(const float* __restrict__ row, int n, int distance) {
  return row[min(max(distance, 0), n - 1)] * 1.4426950408889634f;
}
// the first key that a query at position p sees
__device__ __forceinline__ int first_seen(int p, int window, int chunk) {
  int lo = window > 0 ? max(0, p - window + 1) : 0;
  if (chunk > 0) lo = max(lo, p - p % chunk);
  return lo;
}
// the bias in base-2 units: r1 * log2(1 + r2 * distance); lg2.approx is exact to float32 rounding on [1, inf)
__device__ __forceinline__ float log_distance_bias2(float r1, float r2, int distance) {
  return r1 * __log2f(fmaf(r2, (float)max(distance, 0), 1.0f));
}
// the same for a distance that is a float already: a thread converts one distance per tile and row and steps from it by
// constants, which leaves the logarithm and the exponential as the only special-function operations per score
__device__ __forceinline__ float log_distance_bias2f(float r1, float r2, float distance) {
  return r1 * __log2f(fmaf(r2, fmaxf(distance, 0.f), 1.0f));
}

// Shared-memory stage: TILE rows of K then TILE rows of V (a cache whose keys are its values: TILE rows that serve as both, so
// that the same memory holds twice the stages).  Every row carries 16 bytes of padding, which
// makes the 8 rows of an ldmatrix fall into different banks for any HD.  Head size 64 is the exception: its rows
// are exactly 128 bytes and the 16-byte chunk c of row r sits at chunk c ^ (r & 7) instead, so that a stage is 16 KB
// and three stages leave room for four blocks on an SM (at head size 128 the same layout was measured slower than
// the padding: 108 us against 100 us for 64 requests of 2,048 keys).
template <int HD, int TILE = kTileKeys> struct Stage {
  static constexpr bool kSwizzled = HD == 64;
  static constexpr int kRowBytes = kSwizzled ? HD * 2 : HD * 2 + 16;
  static constexpr int kBytes = 2 * TILE * kRowBytes;
  static constexpr int kChunks = HD / 8;   // 16-byte chunks per row
  // byte offset of chunk `chunk` of row `row` inside the K (or the V) half of a stage
  __device__ static __forceinline__ uint32_t off(int row, int chunk) {
    return (uint32_t)(row * kRowBytes + ((kSwizzled ? (chunk ^ (row & 7)) : chunk) << 4));
  }
};

// Issues the copies of keys [key0, key0 + TILE) of kv head `kvh` into the stage at `stage_base`, by a block of THREADS.
// Keys outside [lo, hi) (and not among the first `keep`) and keys whose page entry is negative are zero-filled, never read.
// A thread copies one 16-byte column of several CONSECUTIVE rows, so that it looks its page up once per
// page rather than once per row; a warp's copies of one pass cover whole rows (coalesced).
// `table` may be a copy of a slice of the request's block table: entry i of it is block i + table_off.
// ONE: the cache holds one vector per token and head; no V half is written.
template <int HD, int TILE = kTileKeys, int THREADS = kThreads, bool ONE = false>
__device__ __forceinline__ void load_stage(uint32_t stage_base, const PagedKV& kv, const int* __restrict__ table, int kvh,
                                           int key0, int lo, int hi, int table_off = 0, int keep = 0) {
  using S = Stage<HD, TILE>;
  const size_t v_off = (size_t)kv.v_off;
  const size_t head_off = (size_t)kvh * kv.block_size * HD;
  const int mask = kv.block_size - 1;
  if constexpr (THREADS % S::kChunks == 0) {
    constexpr int kRowsPerThread = TILE * S::kChunks / THREADS;   // = kChunks / 2
    const int c = threadIdx.x % S::kChunks, row0 = (threadIdx.x / S::kChunks) * kRowsPerThread;
    const bf16* page_ptr = nullptr;
    bool have_page = false;                         // page_ptr belongs to the page of the current row
#pragma unroll
    for (int it = 0; it < kRowsPerThread; ++it) {
      const int row = row0 + it, key = key0 + row, slot = key & mask;
      const bool in_range = (key >= lo || key < keep) && key < hi;
      if (slot == 0) have_page = false;
      if (in_range && !have_page) {
        const int page = table[(key >> kv.block_shift) - table_off];
        page_ptr = page >= 0 ? kv.cache + (size_t)page * kv.page_stride + head_off + c * 8 : nullptr;
        have_page = true;
      }
      const bool ok = in_range && page_ptr != nullptr;
      const bf16* src = ok ? page_ptr + (size_t)slot * HD : kv.cache;
      const uint32_t dst = stage_base + S::off(row, c);
      cp_async_16(dst, src, ok ? 16 : 0);
      if (!ONE) cp_async_16(dst + TILE * S::kRowBytes, ok ? src + v_off : src, ok ? 16 : 0);
    }
  } else {
    static_assert((TILE * S::kChunks) % THREADS == 0, "a stage's copies must divide evenly among the threads");
#pragma unroll
    for (int it = 0; it < (TILE * S::kChunks) / THREADS; ++it) {
      const int idx = threadIdx.x + it * THREADS;
      const int row = idx / S::kChunks, c = idx % S::kChunks;
      const int key = key0 + row;
      const bf16* src = kv.cache;
      int bytes = 0;
      if ((key >= lo || key < keep) && key < hi) {
        const int page = table[(key >> kv.block_shift) - table_off];
        if (page >= 0) {
          src = kv.cache + (size_t)page * kv.page_stride + head_off + (size_t)(key & mask) * HD + c * 8;
          bytes = 16;
        }
      }
      const uint32_t dst = stage_base + S::off(row, c);
      cp_async_16(dst, src, bytes);
      if (!ONE) cp_async_16(dst + TILE * S::kRowBytes, bytes ? src + v_off : src, bytes);
    }
  }
}

}  // namespace fa
}  // namespace lmsf
