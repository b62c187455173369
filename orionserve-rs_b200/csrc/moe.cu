// Mixture of experts: the choice of experts, the order of rows by expert, and the grouped products of the f32 build and of
// sizes the tensor cores do not take (moe_gemm_tc.cu has the others).
//   moe_choose_kernel  one warp per row: sigmoid or softmax scores of the router's logits, the `top` largest (the lower index of equal
//                      ones; where experts form groups, among the best groups), and a histogram per block of rows
//   moe_place_kernel   one warp per row: its places in the order by expert (rows of an expert keep their order, so the order
//                      does not depend on timing), and the row copied there; the first CTA lists the tiles
//   moe_route_kernel   both for up to 64 rows, in one cluster
//   moe_simt_kernel    64 rows x 64 columns of one tile, k ascending, optionally with the gated activation of the scored products
//   moe_swiglu_kernel  the same activation on k-split products (moe_act_kernel: of experts without a gate)
#include "kernels.h"
#include "mma.cuh"

#include <algorithm>

namespace orion {
namespace {

// Rows of one histogram: 8 (a warp each), or 64 in batches whose blocks would otherwise be many.
__host__ __device__ inline uint32_t row_block(uint32_t rows) { return rows <= 512 ? 8 : 64; }
constexpr uint32_t kPlaceRows = 8;
constexpr uint32_t kClusterRows = 64;  // batches of up to this many rows: one kernel, a cluster of a CTA per 8 rows

// The largest of `value(e)` over the warp's n entries and its place, the lower one of equal ones; at = n or more if there is none.
template <typename F>
__device__ __forceinline__ void warp_best(uint32_t n, F value, float &best, uint32_t &at) {
  best = -INFINITY, at = 0xFFFFFFFFu;
  for (uint32_t e = threadIdx.x & 31; e < n; e += 32) {
    const float v = value(e);
    if (v > best) best = v, at = e;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
    const uint32_t oi = __shfl_xor_sync(0xffffffffu, at, o);
    if (ov > best || (ov == best && oi < at)) best = ov, at = oi;
  }
}

// Leaves the scores of the `keep` best groups in `mine` and minus infinity for the others. Scores are not negative, so the sign bit can
// mark the groups that have been taken.
__device__ __forceinline__ void keep_groups(const MoeShape &s, float *mine) {
  const uint32_t lane = threadIdx.x & 31, outputs = s.outputs(), per = outputs / s.groups;
  for (uint32_t k = 0; k < s.keep; ++k) {
    float best;
    uint32_t at;
    warp_best(outputs, [&](uint32_t e) { return signbit(mine[e]) ? -INFINITY : mine[e]; }, best, at);
    __syncwarp();
    if (at >= outputs) break;  // only if scores are not numbers
    const uint32_t first = at / per * per;
    for (uint32_t e = first + lane; e < first + per; e += 32) mine[e] = -mine[e];
    __syncwarp();
  }
  for (uint32_t e = lane; e < outputs; e += 32) mine[e] = signbit(mine[e]) ? -mine[e] : -INFINITY;
  __syncwarp();
}

// One warp: scores of one row in `mine`, its choices to chosen / score, those that name an expert with weights counted in `count`
// (shared memory). The correction takes part in the choice only.
__device__ __forceinline__ void choose_row(const float *__restrict__ logits, uint32_t splits, size_t split_stride,
                                           const float *__restrict__ correction, const MoeShape &s, float *mine, uint32_t *chosen, float *score,
                                           uint32_t *count) {
  const uint32_t lane = threadIdx.x & 31, outputs = s.outputs();
  float most = -INFINITY;
  for (uint32_t e = lane; e < outputs; e += 32) {
    float z = 0.f;
    for (uint32_t s0 = 0; s0 < splits; s0 += 8) {  // eight independent loads in flight
      float x[8];
#pragma unroll
      for (uint32_t s = 0; s < 8; ++s) x[s] = s0 + s < splits ? logits[(s0 + s) * split_stride + e] : 0.f;
#pragma unroll
      for (uint32_t s = 0; s < 8; ++s) z += x[s];
    }
    mine[e] = s.softmax ? z : sigmoid_f(z);
    most = fmaxf(most, z);
  }
  if (s.softmax) {
    most = warp_max(most);
    float sum = 0.f;
    for (uint32_t e = lane; e < outputs; e += 32) sum += mine[e] = expf(mine[e] - most);
    sum = warp_sum(sum);
    for (uint32_t e = lane; e < outputs; e += 32) mine[e] /= sum;
  }
  __syncwarp();
  if (s.groups && s.keep < s.groups) keep_groups(s, mine);
  float total = 0.f, own = 0.f;  // lane k keeps the score of choice k until their sum is known
  for (uint32_t k = 0; k < s.top; ++k) {
    float best;
    uint32_t at;
    warp_best(outputs, [&](uint32_t e) { return correction ? mine[e] + correction[e] : mine[e]; }, best, at);
    if (at >= outputs) at = k;  // only if scores are not numbers: stay inside the router's outputs (top is at most as many)
    __syncwarp();
    if (s.renorm) {
      total += mine[at];
      if (lane == k) own = mine[at];
      __syncwarp();
    }
    if (lane == 0) {
      chosen[k] = at;
      score[k] = mine[at];
      mine[at] = -INFINITY;
      if (at < s.experts) atomicAdd(&count[at], 1u);
    }
    __syncwarp();
  }
  if (s.renorm) {
    for (uint32_t k = 32 + lane; k < s.top; k += 32) score[k] /= total + 1e-20f;
    if (lane < s.top) score[lane] = own / (total + 1e-20f);
    __syncwarp();
  }
}

__global__ void __launch_bounds__(1024)
moe_choose_kernel(const float *__restrict__ logits, uint32_t splits, size_t split_stride, const float *__restrict__ correction, MoeShape s,
                  uint32_t rows, uint32_t *__restrict__ chosen, float *__restrict__ score, uint32_t *__restrict__ histogram) {
  extern __shared__ float smem[];  // [warps][outputs] scores, [experts] counts
  const uint32_t tid = threadIdx.x, warp = tid >> 5, warps = blockDim.x >> 5, block = row_block(rows), experts = s.experts, top = s.top,
                 outputs = s.outputs();
  uint32_t *count = reinterpret_cast<uint32_t *>(smem + warps * outputs);
  pdl_trigger();
  pdl_wait();
  for (uint32_t e = tid; e < experts; e += blockDim.x) count[e] = 0;
  __syncthreads();
  const uint32_t end = min(rows, (blockIdx.x + 1) * block);
  for (uint32_t row = blockIdx.x * block + warp; row < end; row += warps)
    choose_row(logits + (size_t)row * s.row_ld(), splits, split_stride, correction, s, smem + warp * outputs, chosen + (size_t)row * top,
               score + (size_t)row * top, count);
  __syncthreads();
  for (uint32_t e = tid; e < experts; e += blockDim.x) histogram[(size_t)blockIdx.x * experts + e] = count[e];
}

// Exclusive prefix sums of f(value[i]) over `n` values in shared memory, by one warp.
template <typename F>
__device__ __forceinline__ void warp_prefix(const uint32_t *value, uint32_t n, uint32_t *prefix, F f) {
  const uint32_t lane = threadIdx.x & 31;
  uint32_t carry = 0;
  for (uint32_t i0 = 0; i0 < n; i0 += 32) {
    const uint32_t own = i0 + lane < n ? f(value[i0 + lane]) : 0;
    uint32_t v = own;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const uint32_t up = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= (uint32_t)o) v += up;
    }
    if (i0 + lane < n) prefix[i0 + lane] = carry + v - own;
    carry += __shfl_sync(0xffffffffu, v, 31);
  }
}

// The tile list from the rows of every expert (total), their first rows and their first tiles; by a whole CTA.
__device__ __forceinline__ void list_tiles(const uint32_t *total, const uint32_t *first, const uint32_t *tile_at, uint32_t E, uint32_t tile_rows,
                                           uint32_t max_tiles, MoeTile *tiles) {
  for (uint32_t e = threadIdx.x; e < E; e += blockDim.x)
    for (uint32_t t = 0; t * tile_rows < total[e]; ++t)
      if (tile_at[e] + t < max_tiles) tiles[tile_at[e] + t] = MoeTile{e, first[e] + t * tile_rows, min(tile_rows, total[e] - t * tile_rows)};
  const uint32_t used = tile_at[E - 1] + (total[E - 1] + tile_rows - 1) / tile_rows;
  for (uint32_t t = used + threadIdx.x; t < max_tiles; t += blockDim.x) tiles[t] = MoeTile{0, 0, 0};
}

// Copies a row, by one warp.
template <typename T>
__device__ __forceinline__ void copy_row(const T *src, T *dst, uint32_t n) {
  const uint32_t lane = threadIdx.x & 31;
  constexpr uint32_t kVec = 16 / sizeof(T);
  if (n % kVec == 0) {
#pragma unroll 4
    for (uint32_t c = lane; c < n / kVec; c += 32) reinterpret_cast<uint4 *>(dst)[c] = reinterpret_cast<const uint4 *>(src)[c];
  } else {
    for (uint32_t c = lane; c < n; c += 32) dst[c] = src[c];
  }
}

template <typename T>
__global__ void __launch_bounds__(kPlaceRows * 32)
moe_place_kernel(const uint32_t *__restrict__ chosen, const float *__restrict__ score, const uint32_t *__restrict__ histogram,
                 const T *__restrict__ x, MoeShape s, uint32_t rows, uint32_t tile_rows, uint32_t max_tiles, uint32_t *__restrict__ place,
                 float *__restrict__ row_score, MoeTile *__restrict__ tiles, T *__restrict__ sorted) {
  extern __shared__ uint32_t words[];
  uint32_t *total = words, *before = total + s.experts, *first = before + s.experts, *tile_at = first + s.experts;
  pdl_trigger();
  pdl_wait();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = s.experts, top = s.top, per = row_block(rows);
  for (uint32_t e = tid; e < 2 * E; e += blockDim.x) total[e] = 0;  // and `before`
  __syncthreads();
  const uint32_t row0 = blockIdx.x * kPlaceRows, block = row0 / per, blocks = (rows + per - 1) / per;
  for (uint32_t i = tid; i < blocks * E; i += blockDim.x) {
    const uint32_t v = histogram[i], e = i % E;
    if (v == 0) continue;
    atomicAdd(&total[e], v);
    if (i / E < block) atomicAdd(&before[e], v);
  }
  __syncthreads();
  if (warp == 0) warp_prefix(total, E, first, [](uint32_t v) { return v; });
  if (warp == 1 && blockIdx.x == 0) warp_prefix(total, E, tile_at, [&](uint32_t v) { return (v + tile_rows - 1) / tile_rows; });
  __syncthreads();
  if (blockIdx.x == 0) list_tiles(total, first, tile_at, E, tile_rows, max_tiles, tiles);
  const uint32_t row = row0 + warp;
  if (row >= rows) return;
  for (uint32_t k = 0; k < top; ++k) {
    const uint32_t at = row * top + k, e = chosen[at];
    if (e >= E) {  // an identity expert
      if (lane == 0) place[at] = kNoPlace;
      continue;
    }
    uint32_t rank = 0;  // choices of the same expert before this one in the block of rows
    for (uint32_t j = block * per * top; j < at; j += 32) {
      const uint32_t other = j + lane < at ? chosen[j + lane] : 0xFFFFFFFFu;
      rank += __popc(__ballot_sync(0xffffffffu, other == e));
    }
    const uint32_t to = first[e] + before[e] + rank;
    if (lane == 0) {
      place[at] = to;
      row_score[to] = score[at];
    }
    copy_row(x + (size_t)row * s.hidden, sorted + (size_t)to * s.hidden, s.hidden);
  }
}

__device__ __forceinline__ uint32_t ld_dsmem_u32(const uint32_t *local, uint32_t rank) {
  uint32_t addr, v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(smem_u32(local)), "r"(rank));
  asm volatile("ld.shared::cluster.u32 %0, [%1];" : "=r"(v) : "r"(addr) : "memory");
  return v;
}

// Few rows: both steps in one kernel. The CTAs of the one cluster take eight rows each and read each other's counts through
// distributed shared memory.
template <typename T>
__global__ void __launch_bounds__(kPlaceRows * 32)
moe_route_kernel(const float *__restrict__ logits, uint32_t splits, size_t split_stride, const float *__restrict__ correction,
                 const T *__restrict__ x, MoeShape s, uint32_t rows, uint32_t tile_rows, uint32_t max_tiles, uint32_t *__restrict__ place,
                 float *__restrict__ row_score, float *__restrict__ weight, MoeTile *__restrict__ tiles, T *__restrict__ sorted) {
  extern __shared__ float smem[];  // [8][outputs] scores, then words
  const uint32_t E = s.experts, R = s.outputs(), top = s.top, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  uint32_t *count = reinterpret_cast<uint32_t *>(smem + kPlaceRows * R), *total = count + E, *before = total + E, *first = before + E,
           *tile_at = first + E, *chosen = tile_at + E;
  float *score = reinterpret_cast<float *>(chosen + kPlaceRows * top);
  pdl_trigger();
  for (uint32_t e = tid; e < E; e += blockDim.x) count[e] = 0;
  __syncthreads();
  pdl_wait();
  const uint32_t row = blockIdx.x * kPlaceRows + warp;
  if (row < rows)
    choose_row(logits + (size_t)row * s.row_ld(), splits, split_stride, correction, s, smem + warp * R, chosen + warp * top, score + warp * top, count);
  __syncthreads();
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
  for (uint32_t e = tid; e < E; e += blockDim.x) {
    uint32_t all = 0, lower = 0;
    for (uint32_t r = 0; r < gridDim.x; ++r) {
      const uint32_t v = ld_dsmem_u32(count + e, r);
      all += v;
      if (r < blockIdx.x) lower += v;
    }
    total[e] = all, before[e] = lower;
  }
  __syncwarp();
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");  // nobody leaves while its counts may still be read
  __syncthreads();
  if (warp == 0) warp_prefix(total, E, first, [](uint32_t v) { return v; });
  if (warp == 1) warp_prefix(total, E, tile_at, [&](uint32_t v) { return (v + tile_rows - 1) / tile_rows; });
  __syncthreads();
  if (blockIdx.x == 0) list_tiles(total, first, tile_at, E, tile_rows, max_tiles, tiles);
  if (row < rows) {
    for (uint32_t k = 0; k < top; ++k) {
      const uint32_t at = warp * top + k, e = chosen[at];
      if (weight && lane == 0) weight[row * top + k] = score[at];
      if (e >= E) {
        if (lane == 0) place[row * top + k] = kNoPlace;
        continue;
      }
      uint32_t rank = 0;
      for (uint32_t j = 0; j < at; j += 32) {
        const uint32_t other = j + lane < at ? chosen[j + lane] : 0xFFFFFFFFu;
        rank += __popc(__ballot_sync(0xffffffffu, other == e));
      }
      const uint32_t to = first[e] + before[e] + rank;
      if (lane == 0) {
        place[row * top + k] = to;
        row_score[to] = score[at];
      }
      copy_row(x + (size_t)row * s.hidden, sorted + (size_t)to * s.hidden, s.hidden);
    }
  }
  __syncwarp();
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

constexpr uint32_t BM = 64, BN = 64, BK = 16;
template <typename T>
struct SimtFamily {
  const T *x, *w;
  uint32_t n, k;
  T *act;
  float *out;
  GatedAct gate;
};
// ACT: 0 = f32 products, 1 = a gated activation of them, 2 = an activation without a gate.
template <typename T, int ACT>
__global__ void __launch_bounds__(256)
moe_simt_kernel(SimtFamily<T> routed, SimtFamily<T> shared, uint32_t shared_tiles, uint32_t rows, const MoeTile *__restrict__ tiles,
                const float *__restrict__ row_score) {
  __shared__ float xs[BK][BM + 1], ws[BK][BN + 1];
  pdl_trigger();
  pdl_wait();
  const bool is_shared = blockIdx.y < shared_tiles;
  const SimtFamily<T> f = is_shared ? shared : routed;
  MoeTile t;
  if (is_shared) t = MoeTile{0, blockIdx.y * BM, min(BM, rows - blockIdx.y * BM)};
  else t = tiles[blockIdx.y - shared_tiles];
  const uint32_t n0 = blockIdx.x * BN;
  if (t.count == 0 || n0 >= f.n) return;
  const T *w = f.w + (size_t)t.expert * f.n * f.k;
  const uint32_t tx = threadIdx.x % 16, ty = threadIdx.x / 16;
  float acc[4][4] = {};
  for (uint32_t k0 = 0; k0 < f.k; k0 += BK) {
    for (uint32_t idx = threadIdx.x; idx < BM * BK; idx += 256) {
      const uint32_t r = idx / BK, k = k0 + idx % BK;
      xs[idx % BK][r] = r < t.count && k < f.k ? to_f32<T>(f.x[(size_t)(t.row + r) * f.k + k]) : 0.f;
      ws[idx % BK][r] = n0 + r < f.n && k < f.k ? to_f32<T>(w[(size_t)(n0 + r) * f.k + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (uint32_t k = 0; k < BK; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = xs[k][ty * 4 + i], b[i] = ws[k][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t r = ty * 4 + i;
    if (r >= t.count) continue;
    const size_t row = t.row + r;
    const float score = is_shared || !ACT || !row_score ? 1.f : row_score[row];  // multiplies what the expert reads
#pragma unroll
    for (int j = 0; j < 4; j += ACT == 1 ? 2 : 1) {
      const uint32_t n = n0 + tx * 4 + j;
      if (n >= f.n) continue;
      if (ACT == 1) f.act[row * (f.n / 2) + n / 2] = from_f32<T>(gated<T>(f.gate, score * acc[i][j], score * acc[i][j + (ACT == 1 ? 1 : 0)]));
      else if (ACT == 2) f.act[row * f.n + n] = from_f32<T>(gelu_erf<T>(score * acc[i][j]));
      else f.out[row * f.n + n] = acc[i][j];
    }
  }
}

// Products [splits][rows][2 * ffn] with gate and up in neighbouring columns -> act [rows][ffn]; routed rows first.
template <typename T>
__global__ void __launch_bounds__(256)
moe_swiglu_kernel(const float *__restrict__ up, uint32_t splits, MoeShape s, uint32_t rows, const float *__restrict__ row_score, T *__restrict__ act) {
  pdl_trigger();
  pdl_wait();
  const size_t sorted = (size_t)rows * s.top, routed = sorted * s.ffn, all = routed + (size_t)rows * s.shared_ffn;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < all; i += (size_t)gridDim.x * blockDim.x) {
    const bool is_shared = i >= routed;
    const size_t stride = is_shared ? (size_t)rows * 2 * s.shared_ffn : sorted * 2 * s.ffn;
    const float2 *p = reinterpret_cast<const float2 *>(up + (is_shared ? splits * sorted * 2 * s.ffn + 2 * (i - routed) : 2 * i));
    float2 v = make_float2(0.f, 0.f);
    for (uint32_t k = 0; k < splits; ++k) {
      const float2 q = p[k * stride / 2];
      v.x += q.x, v.y += q.y;
    }
    const float w = is_shared || !row_score ? 1.f : row_score[i / s.ffn];
    act[i] = from_f32<T>(gated<T>(is_shared ? s.shared_act : s.act, w * v.x, w * v.y));
  }
}

// The same for experts without a gate: [splits][rows][ffn].
template <typename T>
__global__ void __launch_bounds__(256)
moe_act_kernel(const float *__restrict__ up, uint32_t splits, MoeShape s, uint32_t rows, const float *__restrict__ row_score, T *__restrict__ act) {
  pdl_trigger();
  pdl_wait();
  const size_t routed = (size_t)rows * s.top * s.ffn, all = routed + (size_t)rows * s.shared_ffn;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < all; i += (size_t)gridDim.x * blockDim.x) {
    const bool is_shared = i >= routed;
    const size_t stride = is_shared ? all - routed : routed;
    const float *p = up + (is_shared ? splits * routed + (i - routed) : i);
    float v = 0.f;
    for (uint32_t k = 0; k < splits; ++k) v += p[k * stride];
    act[i] = from_f32<T>(gelu_erf<T>((is_shared || !row_score ? 1.f : row_score[i / s.ffn]) * v));
  }
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

}  // namespace

size_t moe_histogram_words(MoeShape s, uint32_t rows) {
  const uint32_t most = std::max((rows + 63) / 64, (std::min(rows, 512u) + 7) / 8);
  return (size_t)most * s.experts;
}

MoePlan moe_plan(bool is_bf16, MoeShape s, uint32_t rows) {
  MoePlan p{BM, 0, 1, 1, is_bf16 && moe_tc_supported(s)};
  const uint64_t choices = (uint64_t)rows * s.top;
  if (p.tensor_core) {
    // Few rows: one tile holds every row of an expert and all rows of the shared one. More: by the mean rows of an expert.
    const uint64_t mean = (choices + s.experts - 1) / s.experts;
    p.tile_rows = rows <= 16 ? 16 : (rows <= 32 ? 32 : (rows <= 64 || mean <= 48 ? 64 : (mean <= 160 ? 128 : 256)));
  }
  const uint64_t busy = std::min<uint64_t>(s.experts, choices);  // experts that have rows, at most
  p.tiles = (uint32_t)(busy + choices / p.tile_rows);
  if (p.tensor_core && rows <= 64) {
    // k splits until a wave of two CTAs per SM is full, at least four k slabs each
    auto splits = [&](uint32_t n, uint32_t shared_n, uint32_t k) {
      const uint64_t ctas = busy * ((n + 127) / 128) + (shared_n + 127) / 128;
      const uint32_t most = std::max(1u, (k + 63) / 64 / 4);
      return (uint32_t)std::max<uint64_t>(1, std::min<uint64_t>({296 / std::max<uint64_t>(1, ctas), most, 8}));
    };
    p.up_splits = splits(s.up_cols(), s.shared_up_cols(), s.hidden);
    p.down_splits = splits(s.hidden, s.shared_ffn ? s.hidden : 0, s.ffn);
  }
  return p;
}

size_t moe_up_floats(bool is_bf16, MoeShape s, uint32_t rows) {
  const MoePlan p = moe_plan(is_bf16, s, rows);
  return p.up_splits == 1 ? 0 : (size_t)p.up_splits * rows * ((size_t)s.top * s.up_cols() + s.shared_up_cols());
}

template <typename T>
int launch_moe_route(const float *logits, uint32_t splits, size_t split_stride, const float *correction, const T *x, MoeShape s, MoePlan plan,
                     MoeBuffers<T> b, uint32_t rows, cudaStream_t stream) {
  if (rows == 0) return ORION_OK;
  const uint32_t outputs = s.outputs();
  if (s.experts == 0 || outputs > kMoeMaxExperts || s.top == 0 || s.top > outputs)
    return set_error(ORION_ERR_INTERNAL, "routing of %u among %u experts is not supported (at most %u)", s.top, outputs, kMoeMaxExperts);
  if (s.groups && (!s.softmax || correction || outputs % s.groups || s.keep == 0 || s.keep > s.groups || s.top > outputs / s.groups * s.keep))
    return set_error(ORION_ERR_INTERNAL, "routing of %u among %u of %u groups of %u experts is not supported", s.top, s.keep, s.groups, outputs);
  if (rows <= kClusterRows) {
    const uint32_t ctas = (rows + kPlaceRows - 1) / kPlaceRows;
    const size_t smem = (kPlaceRows * (size_t)outputs + 5 * (size_t)s.experts + 2 * kPlaceRows * s.top) * 4;
    static bool attr_set[kMaxDeviceOrdinals] = {};
    ORION_CUDA_CHECK("moe_route attr", ensure_dynamic_smem(moe_route_kernel<T>, ((kPlaceRows + 5) + 2 * kPlaceRows) * kMoeMaxExperts * 4, attr_set));
    ORION_CUDA_CHECK("moe_route", launch_pdl_cluster(moe_route_kernel<T>, dim3(ctas), dim3(kPlaceRows * 32), dim3(ctas), smem, stream, logits, splits,
                                                     split_stride, correction, x, s, rows, plan.tile_rows, plan.tiles, b.place, b.row_score,
                                                     s.weigh_output ? b.score : nullptr, b.tiles, b.x));
    return after_launch("moe_route");
  }
  const uint32_t block = row_block(rows), threads = block == 8 ? 256 : 1024;
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("moe_choose attr", ensure_dynamic_smem(moe_choose_kernel, 33 * kMoeMaxExperts * (int)sizeof(float), attr_set));
  ORION_CUDA_CHECK("moe_choose", launch_pdl(moe_choose_kernel, dim3((rows + block - 1) / block), dim3(threads),
                                            (threads / 32 * outputs + s.experts) * sizeof(float), stream, logits, splits, split_stride, correction, s,
                                            rows, b.chosen, b.score, b.histogram));
  ORION_TRY(after_launch("moe_choose"));
  ORION_CUDA_CHECK("moe_place", launch_pdl(moe_place_kernel<T>, dim3((rows + kPlaceRows - 1) / kPlaceRows), dim3(kPlaceRows * 32),
                                           4 * s.experts * sizeof(uint32_t), stream, b.chosen, b.score, b.histogram, x, s, rows, plan.tile_rows,
                                           plan.tiles, b.place, b.row_score, b.tiles, b.x));
  return after_launch("moe_place");
}

namespace {
template <typename T>
int launch_simt(int act, SimtFamily<T> routed, SimtFamily<T> shared, MoePlan plan, const MoeBuffers<T> &b, const float *row_score, uint32_t rows,
                cudaStream_t stream) {
  const uint32_t shared_tiles = shared.n ? (rows + BM - 1) / BM : 0;
  const dim3 grid((std::max(routed.n, shared.n) + BN - 1) / BN, shared_tiles + plan.tiles);
  auto kernel = act == 0 ? moe_simt_kernel<T, 0> : (act == 1 ? moe_simt_kernel<T, 1> : moe_simt_kernel<T, 2>);
  ORION_CUDA_CHECK("moe_simt", launch_pdl(kernel, grid, dim3(256), 0, stream, routed, shared, shared_tiles, rows, (const MoeTile *)b.tiles,
                                          row_score));
  return after_launch("moe_simt");
}
}  // namespace

template <typename T>
int launch_moe_experts(const T *x, const T *w_up, const T *w_down, const T *shared_up, const T *shared_down, MoeShape s, MoePlan plan,
                       MoeBuffers<T> b, float *shared_out, uint32_t rows, cudaStream_t stream) {
  if (rows == 0) return ORION_OK;
  const size_t sorted = (size_t)rows * s.top;
  const float *row_score = s.weigh_output ? nullptr : b.row_score;
  T *shared_act = b.act + sorted * s.ffn;
  const uint32_t up_n = s.up_cols(), shared_up_n = s.shared_up_cols();
  if (s.act.plain() != s.shared_act.plain()) return set_error(ORION_ERR_INTERNAL, "routed and shared experts are of one form");
  if constexpr (sizeof(T) == 2) {
    if (plan.tensor_core) {
      const bool fused = plan.up_splits == 1;
      float *shared_up_out = fused ? nullptr : b.up + plan.up_splits * sorted * up_n;
      MoeProduct p{b.x, w_up, x, shared_up, up_n, s.hidden, shared_up_n, s.hidden, (uint32_t)sorted, rows, s.experts, b.tiles, row_score,
                   b.act, shared_act, fused ? nullptr : b.up, shared_up_out, s.act, s.shared_act};
      ORION_TRY(launch_moe_product_tc(p, fused, plan.up_splits, plan, stream));
      if (!fused) {
        const size_t n = sorted * s.ffn + (size_t)rows * s.shared_ffn;
        ORION_CUDA_CHECK("moe_swiglu", launch_pdl(s.act.plain() ? moe_act_kernel<T> : moe_swiglu_kernel<T>, dim3((uint32_t)std::min<size_t>((n + 255) / 256, 148 * 8)), dim3(256), 0, stream,
                                                  (const float *)b.up, plan.up_splits, s, rows, row_score, b.act));
        ORION_TRY(after_launch("moe_swiglu"));
      }
      MoeProduct d{b.act, w_down, shared_act, shared_down, s.hidden, s.ffn, s.shared_ffn ? s.hidden : 0, s.shared_ffn, (uint32_t)sorted, rows, s.experts,
                   b.tiles, nullptr, nullptr, nullptr, b.down, shared_out};
      return launch_moe_product_tc(d, false, plan.down_splits, plan, stream);
    }
  }
  ORION_TRY(launch_simt<T>(s.act.plain() ? 2 : 1, {b.x, w_up, up_n, s.hidden, b.act, nullptr, s.act},
                           {x, shared_up, shared_up_n, s.hidden, shared_act, nullptr, s.shared_act}, plan, b, row_score, rows, stream));
  return launch_simt<T>(0, {b.act, w_down, s.hidden, s.ffn, nullptr, b.down},
                        {shared_act, shared_down, s.shared_ffn ? s.hidden : 0, s.shared_ffn, nullptr, shared_out}, plan, b, nullptr, rows, stream);
}

#define ORION_INSTANTIATE(T)                                                                                                            \
  template int launch_moe_route<T>(const float *, uint32_t, size_t, const float *, const T *, MoeShape, MoePlan, MoeBuffers<T>, uint32_t, cudaStream_t); \
  template int launch_moe_experts<T>(const T *, const T *, const T *, const T *, const T *, MoeShape, MoePlan, MoeBuffers<T>, float *,    \
                                     uint32_t, cudaStream_t);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
