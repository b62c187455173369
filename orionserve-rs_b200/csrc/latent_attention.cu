// Latent attention: queries and keys meet in a per-head space that is a linear image of one small latent per
// token, plus one rotated key part shared by all heads; only the latent and the shared part are cached. The
// product with a key is evaluated in the latent space: q . (W_uk c) = (W_uk^T q) . c, and the weighted sum of
// values is W_uv applied to the weighted sum of latents, so a decode step reads the cache once for all heads.
//   latent_prepare_kernel            folds the joint projection: queries rotated, latent normalised and cached
//   latent_attention_generic_kernel  any shape and batch, f32 arithmetic: the f32 build and unusual shapes
//   latent_absorb_kernel             rows that decode: their queries taken into the latent space, per head
//                                    (W_uk^T q on mma.sync)
//   latent_decode_kernel             rows that decode: scores and weighted latents over the window's cache rows
//   latent_value_kernel              rows that decode: merges the context splits, W_uv per head, output gate (if the design has one)
#include "kernels.h"
#include "mma.cuh"

#include <algorithm>

namespace orion {
namespace {

__device__ __forceinline__ float fold(const float *p, uint32_t splits, size_t stride) {
  float v = p[0];
  for (uint32_t s = 1; s < splits; ++s) v += p[s * stride];
  return v;
}

constexpr uint32_t kPrepThreads = 256;

// One CTA per row. Pair i of a rotated part is (2i, 2i + 1); the table holds rope_dims / 2 angles per position.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
latent_prepare_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const float *__restrict__ norm_w,
                      const float *__restrict__ rope_cos, const float *__restrict__ rope_sin, const uint32_t *__restrict__ positions,
                      const uint32_t *__restrict__ slot_block, const uint32_t *__restrict__ slot_slot, T *__restrict__ q,
                      T *__restrict__ cache, LatentShape ls) {
  __shared__ float red[kPrepThreads / 32];
  pdl_trigger();
  const uint32_t row = blockIdx.x, tid = threadIdx.x;
  const uint32_t half = ls.rope_dims / 2;
  const float *cs = rope_cos + (size_t)positions[row] * half, *sn = rope_sin + (size_t)positions[row] * half;
  pdl_wait();
  const float *p = partial + (size_t)row * ls.row_ld();
  // value `i` of a rotated part whose first column is `at`
  auto rotated = [&](const float *at, uint32_t i) {
    const float v = fold(at + i, splits, split_stride);
    if (i >= 2 * half) return v;
    const float other = fold(at + (i ^ 1), splits, split_stride), c = cs[i >> 1], s = sn[i >> 1];
    return (i & 1) ? v * c + other * s : v * c - other * s;
  };
  const uint32_t nq = ls.q_cols(), qd = ls.q_dim();
  for (uint32_t i = tid; i < nq; i += kPrepThreads) {
    const uint32_t d = i % qd;
    const float v = d < ls.dim ? fold(p + i, splits, split_stride) : rotated(p + (i - d + ls.dim), d - ls.dim);
    q[(size_t)row * nq + i] = from_f32<T>(v);
  }
  const float *lat = p + nq;
  T *dst = cache + ((size_t)slot_block[row] * ls.block_size + slot_slot[row]) * ls.row_stride;
  float ss = 0.f;
  for (uint32_t i = tid; i < ls.kv_rank; i += kPrepThreads) {
    const float v = fold(lat + i, splits, split_stride);
    ss += v * v;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (uint32_t w = 0; w < kPrepThreads / 32; ++w) total += red[w];
  const float scale = 1.0f / sqrtf(total / (float)ls.kv_rank + ls.eps);
  for (uint32_t i = tid; i < ls.kv_rank; i += kPrepThreads)
    dst[i] = from_f32<T>(fold(lat + i, splits, split_stride) * scale * norm_w[i]);
  for (uint32_t i = tid; i < ls.rot_dim; i += kPrepThreads) dst[ls.kv_rank + i] = from_f32<T>(rotated(lat + ls.kv_rank, i));
}

// The same, four columns per thread and one round of loads: every part a multiple of four columns. blockIdx.y = 0
// is the row's latent and shared key part, the others are 1024 query columns each.
template <typename T>
__device__ __forceinline__ void store4(T *p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
template <>
__device__ __forceinline__ void store4<bf16>(bf16 *p, float4 v) {
  uint2 x;
  x.x = pack_bf16x2(v.x, v.y);
  x.y = pack_bf16x2(v.z, v.w);
  *reinterpret_cast<uint2 *>(p) = x;
}
__device__ __forceinline__ float4 rotate4(float4 v, float2 c, float2 s) {  // two neighbouring pairs
  return make_float4(v.x * c.x - v.y * s.x, v.y * c.x + v.x * s.x, v.z * c.y - v.w * s.y, v.w * c.y + v.z * s.y);
}

template <typename T>
__global__ void __launch_bounds__(kPrepThreads)
latent_prepare_vec_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const float *__restrict__ norm_w,
                          const float *__restrict__ rope_cos, const float *__restrict__ rope_sin, const uint32_t *__restrict__ positions,
                          const uint32_t *__restrict__ slot_block, const uint32_t *__restrict__ slot_slot, T *__restrict__ q,
                          T *__restrict__ cache, LatentShape ls) {
  __shared__ float red[kPrepThreads / 32];
  pdl_trigger();
  const uint32_t row = blockIdx.x, tid = threadIdx.x, half = ls.rope_dims / 2;
  const float *cs = rope_cos + (size_t)positions[row] * half, *sn = rope_sin + (size_t)positions[row] * half;
  const float *p = partial + (size_t)row * ls.row_ld();
  if (blockIdx.y > 0) {
    const uint32_t i = ((blockIdx.y - 1) * kPrepThreads + tid) * 4, d = i % ls.q_dim();
    const bool live = i < ls.q_cols(), rot = live && d >= ls.dim && d - ls.dim < ls.rope_dims;
    float2 c, sv;
    if (rot) {  // rope_dims is a multiple of 4 here
      c = *reinterpret_cast<const float2 *>(cs + (d - ls.dim) / 2);
      sv = *reinterpret_cast<const float2 *>(sn + (d - ls.dim) / 2);
    }
    pdl_wait();
    if (!live) return;
    float4 v = sum_slabs4(p + i, splits, split_stride);
    if (rot) v = rotate4(v, c, sv);
    store4<T>(q + (size_t)row * ls.q_cols() + i, v);
    return;
  }
  const float *lat = p + ls.q_cols();
  T *dst = cache + ((size_t)slot_block[row] * ls.block_size + slot_slot[row]) * ls.row_stride;
  const uint32_t i = tid * 4;
  pdl_wait();
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (i < ls.kv_cols()) v = sum_slabs4(lat + i, splits, split_stride);
  float ss = i < ls.kv_rank ? v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w : 0.f;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float total = 0.f;
#pragma unroll
  for (uint32_t w = 0; w < kPrepThreads / 32; ++w) total += red[w];
  if (i >= ls.kv_cols()) return;
  if (i < ls.kv_rank) {
    const float scale = 1.0f / sqrtf(total / (float)ls.kv_rank + ls.eps);
    const float4 g = *reinterpret_cast<const float4 *>(norm_w + i);
    v = make_float4(v.x * scale * g.x, v.y * scale * g.y, v.z * scale * g.z, v.w * scale * g.w);
  } else if (i - ls.kv_rank < ls.rope_dims) {
    v = rotate4(v, *reinterpret_cast<const float2 *>(cs + (i - ls.kv_rank) / 2), *reinterpret_cast<const float2 *>(sn + (i - ls.kv_rank) / 2));
  }
  store4<T>(dst + i, v);
}

constexpr uint32_t kGenThreads = 128, kGenKeys = 256;

template <typename T>
__global__ void __launch_bounds__(kGenThreads)
latent_attention_generic_kernel(const T *__restrict__ q, const T *__restrict__ cache, const T *__restrict__ w_uk,
                                const T *__restrict__ w_uv, const float *__restrict__ gate, uint32_t splits, size_t split_stride,
                                LatentShape ls, AttnBatch batch, T *__restrict__ out, uint32_t ldo) {
  extern __shared__ float gen_smem[];
  float *q_s = gen_smem;                     // [kv_rank + rot_dim]: the query in the latent space, then its rotated part
  float *acc = q_s + ls.kv_cols();       // [kv_rank]
  float *scores = acc + ls.kv_rank;      // [kGenKeys]
  __shared__ float red[kGenThreads / 32];
  pdl_trigger();
  pdl_wait();
  const uint32_t row = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t pos = batch.query_positions[row];
  const uint32_t *table = batch.tables_flat + batch.table_offsets[batch.seq_of_row[row]];
  const T *qr = q + (size_t)row * ls.q_cols() + head * ls.q_dim();
  for (uint32_t r = tid; r < ls.kv_rank; r += kGenThreads) {
    float a = 0.f;
    for (uint32_t d = 0; d < ls.dim; ++d) a += to_f32<T>(w_uk[((size_t)head * ls.dim + d) * ls.kv_rank + r]) * to_f32<T>(qr[d]);
    q_s[r] = a;
    acc[r] = 0.f;
  }
  for (uint32_t i = tid; i < ls.rot_dim; i += kGenThreads) q_s[ls.kv_rank + i] = to_f32<T>(qr[ls.dim + i]);
  __syncthreads();

  auto key = [&](uint32_t p) { return cache + ((size_t)table[p / ls.block_size] * ls.block_size + p % ls.block_size) * ls.row_stride; };
  float m = -INFINITY, l = 0.f;
  for (uint32_t k0 = ls.first_key(pos); k0 <= pos; k0 += kGenKeys) {
    const uint32_t n = min(kGenKeys, pos + 1 - k0);
    for (uint32_t i = warp; i < n; i += kGenThreads / 32) {  // one warp per key
      const T *k = key(k0 + i);
      float dot = 0.f;
      for (uint32_t d = lane; d < ls.kv_cols(); d += 32) dot += q_s[d] * to_f32<T>(k[d]);
      dot = warp_sum(dot);
      if (lane == 0) scores[i] = dot * ls.scale;
    }
    __syncthreads();
    float mx = -INFINITY;
    for (uint32_t i = lane; i < n; i += 32) mx = fmaxf(mx, scores[i]);
    mx = fmaxf(m, warp_max(mx));  // the same in every warp
    const float corr = m == -INFINITY ? 0.f : expf(m - mx);
    __syncthreads();
    float sum = 0.f;
    for (uint32_t i = tid; i < n; i += kGenThreads) {
      const float e = expf(scores[i] - mx);
      scores[i] = e;
      sum += e;
    }
    sum = warp_sum(sum);
    if (lane == 0) red[warp] = sum;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (uint32_t w = 0; w < kGenThreads / 32; ++w) total += red[w];
    l = l * corr + total;
    for (uint32_t r = tid; r < ls.kv_rank; r += kGenThreads) {
      float a = acc[r] * corr;
      for (uint32_t i = 0; i < n; ++i) a += scores[i] * to_f32<T>(key(k0 + i)[r]);
      acc[r] = a;
    }
    m = mx;
    __syncthreads();
  }
  const float inv = 1.0f / l;
  const float *g = gate + (size_t)row * ls.row_ld() + ls.q_cols() + ls.kv_cols() + (size_t)head * ls.value_dim;
  T *o = out + (size_t)row * ldo + (size_t)head * ls.value_dim;
  for (uint32_t v = warp; v < ls.value_dim; v += kGenThreads / 32) {
    const T *w = w_uv + ((size_t)head * ls.value_dim + v) * ls.kv_rank;
    float a = 0.f;
    for (uint32_t r = lane; r < ls.kv_rank; r += 32) a += to_f32<T>(w[r]) * acc[r];
    a = warp_sum(a);
    if (lane == 0) o[v] = from_f32<T>(ls.gated ? a * inv * sigmoid_f(fold(g + v, splits, split_stride)) : a * inv);
  }
}

// ---------------------------------------------------------------------------
// Rows that decode (bf16)
// ---------------------------------------------------------------------------

__device__ uint32_t g_latent_error = 0;  // bit 0: a ring wait ran out

constexpr uint32_t kRowTile = 32;  // batch rows per CTA of the per-head products

__device__ __forceinline__ void cp_async16(void *smem, const void *gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// CTA (x: head and 64-wide tile of the latent; y: tile of 32 listed rows).
// A = W_uk of the head, [dim][64 latent columns] (transposed on the way into the fragments), B = the rows' queries.
constexpr uint32_t kAbsorbTile = 64;
__global__ void __launch_bounds__(128)
latent_absorb_kernel(const bf16 *__restrict__ q, const bf16 *__restrict__ w_uk, const uint32_t *__restrict__ row_list, uint32_t rows,
                     bf16 *__restrict__ qa, LatentShape ls) {
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t w_pitch = kAbsorbTile * 2 + 16, q_pitch = ls.dim * 2 + 16;
  uint8_t *w_s = smem, *q_s = smem + ls.dim * w_pitch;
  pdl_trigger();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t tiles = (ls.kv_rank + kAbsorbTile - 1) / kAbsorbTile;
  const uint32_t row0 = blockIdx.y * kRowTile, n = min(kRowTile, rows - row0), qd = ls.q_dim(), width = ls.kv_cols();
  const uint32_t head = blockIdx.x / tiles, r0 = (blockIdx.x % tiles) * kAbsorbTile;
  const uint32_t cols = min(kAbsorbTile, ls.kv_rank - r0);  // a multiple of 16
  for (uint32_t i = tid; i < ls.dim * (cols / 8); i += 128) {
    const uint32_t d = i / (cols / 8), c = i % (cols / 8);
    cp_async16(w_s + d * w_pitch + c * 16, w_uk + ((size_t)head * ls.dim + d) * ls.kv_rank + r0 + c * 8);
  }
  pdl_wait();
  const uint32_t groups = ls.dim / 8;
  for (uint32_t i = tid; i < n * groups; i += 128)  // rows beyond n stay undefined and are not stored
    cp_async16(q_s + (i / groups) * q_pitch + (i % groups) * 16, q + (size_t)row_list[row0 + i / groups] * ls.q_cols() + head * qd + (i % groups) * 8);
  if (r0 == 0) {  // the rotated part goes along with the first tile
    const uint32_t rg = ls.rot_dim / 8;
    for (uint32_t i = tid; i < n * rg; i += 128)
      *reinterpret_cast<uint4 *>(qa + ((size_t)(row0 + i / rg) * ls.heads + head) * width + ls.kv_rank + (i % rg) * 8) =
          *reinterpret_cast<const uint4 *>(q + (size_t)row_list[row0 + i / rg] * ls.q_cols() + head * qd + ls.dim + (i % rg) * 8);
  }
  cp_async_wait_all();
  __syncthreads();
  // warp = 16 latent columns (M), all 32 rows (four n-tiles)
  if (warp * 16 >= cols) return;
  float c[kRowTile / 8][4];
#pragma unroll
  for (uint32_t t = 0; t < kRowTile / 8; ++t) c[t][0] = c[t][1] = c[t][2] = c[t][3] = 0.f;
  const uint32_t mi = lane >> 3, rr = lane & 7;
  const uint32_t wa = smem_u32(w_s) + (rr + (mi >> 1) * 8) * w_pitch + (warp * 16 + (mi & 1) * 8) * 2;
  const uint32_t qb = smem_u32(q_s) + (rr + (mi >> 1) * 8) * q_pitch + (mi & 1) * 16;
  for (uint32_t k = 0; k < ls.dim; k += 16) {
    uint32_t a[4];
    ldmatrix_x4_trans(a, wa + k * w_pitch);
#pragma unroll
    for (uint32_t t = 0; t < kRowTile / 16; ++t) {
      uint32_t b[4];  // rows 16t..+7 (k halves 0, 1), rows 16t+8..+15
      ldmatrix_x4(b, qb + t * 16 * q_pitch + k * 2);
      mma_bf16_16816(c[2 * t], a, b[0], b[1]);
      mma_bf16_16816(c[2 * t + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (uint32_t t = 0; t < kRowTile / 8; ++t)
#pragma unroll
    for (uint32_t e = 0; e < 4; ++e) {
      const uint32_t r = t * 8 + (lane & 3) * 2 + (e & 1), col = r0 + warp * 16 + (lane >> 2) + (e >> 1) * 8;
      if (r < n) qa[((size_t)(row0 + r) * ls.heads + head) * width + col] = __float2bfloat16_rn(c[t][e]);
    }
}

// Scores and weighted latents of one row over one piece of its window, for 8 * NT heads. 64 keys per tile; each
// of the 8 warps scores 32 of them over a quarter of the dimensions with its share of the queries held in
// registers (keys on M, heads on N), the quarters are summed in shared memory, one group of eight lanes per
// head keeps the running maximum and sum, and each warp then accumulates its own 16-wide slices of the weighted
// latent. The cache comes in whole blocks, one bulk copy each, two tiles deep; a row is an odd number of 16-byte
// groups long (LatentShape::row_stride), so the fragments load without bank conflicts.
constexpr uint32_t kTileKeys = 64, kCacheBlock = 16, kTileBlocks = kTileKeys / kCacheBlock, kDecThreads = 256, kDecStages = 2;
constexpr uint32_t kScorePitch = kTileKeys + 8;  // floats
constexpr uint32_t kProbPitch = kTileKeys + 8;   // bf16
struct DecodeSmem {
  uint32_t pitch, ring, scores, probs, stats, bars, total;
  __host__ __device__ DecodeSmem(uint32_t row_stride, uint32_t heads) {
    pitch = row_stride * 2;
    ring = 0;
    scores = ring + kDecStages * kTileKeys * pitch;
    probs = scores + 4 * heads * kScorePitch * 4;
    stats = probs + heads * kProbPitch * 2;
    bars = stats + heads * 4;
    total = bars + 64;
  }
};

template <int NT, int KQ, int MT>
__global__ void __launch_bounds__(kDecThreads)
latent_decode_kernel(const bf16 *__restrict__ qa, const bf16 *__restrict__ cache, const uint32_t *__restrict__ row_list,
                     const uint32_t *__restrict__ first_row, AttnBatch batch, uint32_t splits, float *__restrict__ part_o,
                     float *__restrict__ part_ml, LatentShape ls) {
  constexpr uint32_t kHeads = 8 * NT;
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t width = ls.kv_cols();
  const DecodeSmem lay(ls.row_stride, kHeads);
  float *sS = reinterpret_cast<float *>(smem + lay.scores);
  uint8_t *sP = smem + lay.probs;
  float *sC = reinterpret_cast<float *>(smem + lay.stats);
  uint64_t *full = reinterpret_cast<uint64_t *>(smem + lay.bars);
  pdl_trigger();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t head0 = blockIdx.x * kHeads, item = blockIdx.y, split = blockIdx.z;
  const uint32_t row = row_list[item], pos = batch.query_positions[row], seq = batch.seq_of_row[row];
  const uint32_t *table = batch.tables_flat + batch.table_offsets[seq];
  // tiles start at block borders; keys before the window or past the row's own position are masked
  const uint32_t lo = ls.first_key(pos), block0 = lo / kCacheBlock, last_block = pos / kCacheBlock;
  const uint32_t all_tiles = (last_block - block0) / kTileBlocks + 1;
  const uint32_t per = (all_tiles + splits - 1) / splits;
  const uint32_t t_begin = min(split * per, all_tiles), ntiles = min(per, all_tiles - t_begin);
  const uint32_t my_block0 = block0 + t_begin * kTileBlocks, key0 = my_block0 * kCacheBlock;
  if (tid < kDecStages) mbar_init(&full[tid], 1);
  mbar_fence_init();
  __syncthreads();

  const uint32_t block_bytes = kCacheBlock * lay.pitch;
  auto issue = [&](uint32_t t) {  // warp 0
    uint64_t *bar = &full[t % kDecStages];
    if (lane == 0) mbar_arrive_expect_tx(bar, kTileBlocks * block_bytes);
    __syncwarp();
    if (lane < kTileBlocks) {  // blocks past the end repeat the last one and are masked
      const uint32_t b = min(my_block0 + t * kTileBlocks + lane, last_block);
      bulk_copy_g2s(smem + lay.ring + ((t % kDecStages) * kTileBlocks + lane) * block_bytes,
                    cache + (size_t)table[b] * kCacheBlock * ls.row_stride, block_bytes, bar);
    }
  };
  // tiles that hold no row of this step are fetched before the kernel that writes those rows has finished
  const uint32_t step_first = batch.query_positions[first_row[seq]];
  uint32_t issued = 0;
  if (warp == 0)
    while (issued < min(ntiles, kDecStages) && key0 + (issued + 1) * kTileKeys <= step_first) issue(issued++);
  pdl_wait();
  if (warp == 0)
    while (issued < min(ntiles, kDecStages)) issue(issued++);

  // queries of this warp's quarter of the dimensions (16-wide steps quarter + 4 k) as B fragments
  const uint32_t quarter = warp & 3, key_half = warp >> 2, steps = width / 16;
  uint32_t qf[KQ][NT][2];
#pragma unroll
  for (int k = 0; k < KQ; ++k)
#pragma unroll
    for (int t = 0; t < NT; ++t) {
      const uint32_t h = head0 + t * 8 + (lane >> 2), s = quarter + 4 * k;
      qf[k][t][0] = qf[k][t][1] = 0u;
      if (h < ls.heads && s < steps) {
        const bf16 *src = qa + ((size_t)item * ls.heads + h) * width + s * 16 + (lane & 3) * 2;
        qf[k][t][0] = *reinterpret_cast<const uint32_t *>(src);
        qf[k][t][1] = *reinterpret_cast<const uint32_t *>(src + 8);
      }
    }
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t) o[m][t][0] = o[m][t][1] = o[m][t][2] = o[m][t][3] = 0.f;
  // running maximum (log2 units) and sum of head `sh`, kept alike by the eight lanes of its group
  const uint32_t sh = warp * 4 + (lane >> 3), sl = lane & 7;
  const bool scorer = sh < kHeads;
  float mx = -INFINITY, sum = 0.f;
  const float sl2 = ls.scale * 1.4426950408889634f;
  const uint32_t mi = lane >> 3, rr = lane & 7;
  bool ok = true;

  for (uint32_t t = 0; t < ntiles; ++t) {
    const uint32_t stage = t % kDecStages;
    if (!mbar_wait(&full[stage], (t / kDecStages) & 1)) ok = false;  // no break: the barriers below stay matched
    const uint32_t base = smem_u32(smem + lay.ring) + stage * kTileKeys * lay.pitch;
    {
      float s[2][NT][4];
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n) s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f;
#pragma unroll
      for (int k = 0; k < KQ; ++k) {
        const uint32_t st = quarter + 4 * k;
        if (st < steps) {
#pragma unroll
          for (int m = 0; m < 2; ++m) {
            uint32_t a[4];
            ldmatrix_x4(a, base + (key_half * 32 + m * 16 + rr + (mi & 1) * 8) * lay.pitch + st * 32 + (mi >> 1) * 16);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(s[m][n], a, qf[k][n][0], qf[k][n][1]);
          }
        }
      }
      float *dst = sS + (size_t)quarter * kHeads * kScorePitch;
#pragma unroll
      for (int m = 0; m < 2; ++m)
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            dst[(n * 8 + (lane & 3) * 2 + (e & 1)) * kScorePitch + key_half * 32 + m * 16 + (lane >> 2) + (e >> 1) * 8] = s[m][n][e];
    }
    __syncthreads();
    if (scorer) {
      const uint32_t tile_key = key0 + t * kTileKeys;
      float v[kTileKeys / 8], tm = -INFINITY;
#pragma unroll
      for (uint32_t i = 0; i < kTileKeys / 8; ++i) {
        const uint32_t key = i * 8 + sl;
        const float *p = sS + sh * kScorePitch + key;
        const float x = (p[0] + p[kHeads * kScorePitch]) + (p[2 * kHeads * kScorePitch] + p[3 * kHeads * kScorePitch]);
        v[i] = tile_key + key >= lo && tile_key + key <= pos ? x * sl2 : -INFINITY;
        tm = fmaxf(tm, v[i]);
      }
#pragma unroll
      for (int off = 1; off < 8; off <<= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, off));
      const float nm = fmaxf(mx, tm), corr = fast_exp2(mx - nm);  // finite: every tile holds a key that is seen
      float part = 0.f;
#pragma unroll
      for (uint32_t i = 0; i < kTileKeys / 8; ++i) {
        const float p = fast_exp2(v[i] - nm);
        part += p;
        *reinterpret_cast<bf16 *>(sP + (sh * kProbPitch + i * 8 + sl) * 2) = __float2bfloat16_rn(p);
      }
#pragma unroll
      for (int off = 1; off < 8; off <<= 1) part += __shfl_xor_sync(0xffffffffu, part, off);
      sum = sum * corr + part;
      mx = nm;
      if (sl == 0) sC[sh] = corr;
    }
    __syncthreads();
    {
      float cr[NT][2];
#pragma unroll
      for (int n = 0; n < NT; ++n) cr[n][0] = sC[n * 8 + (lane & 3) * 2], cr[n][1] = sC[n * 8 + (lane & 3) * 2 + 1];
      uint32_t pb[kTileKeys / 16][NT][2];
#pragma unroll
      for (uint32_t k = 0; k < kTileKeys / 16; ++k)
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          const uint8_t *p = sP + ((n * 8 + (lane >> 2)) * kProbPitch + k * 16 + (lane & 3) * 2) * 2;
          pb[k][n][0] = *reinterpret_cast<const uint32_t *>(p);
          pb[k][n][1] = *reinterpret_cast<const uint32_t *>(p + 16);
        }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const uint32_t d0 = (warp + 8 * m) * 16;
        if (d0 < ls.kv_rank) {
#pragma unroll
          for (int n = 0; n < NT; ++n) o[m][n][0] *= cr[n][0], o[m][n][1] *= cr[n][1], o[m][n][2] *= cr[n][0], o[m][n][3] *= cr[n][1];
#pragma unroll
          for (uint32_t k = 0; k < kTileKeys / 16; ++k) {
            uint32_t a[4];
            ldmatrix_x4_trans(a, base + (k * 16 + rr + (mi >> 1) * 8) * lay.pitch + d0 * 2 + (mi & 1) * 16);
#pragma unroll
            for (int n = 0; n < NT; ++n) mma_bf16_16816(o[m][n], a, pb[k][n][0], pb[k][n][1]);
          }
        }
      }
    }
    __syncthreads();  // the stage and the score buffers are free again
    if (warp == 0 && t + kDecStages < ntiles) issue(t + kDecStages);
  }
  if (!ok && lane == 0) atomicOr(&g_latent_error, 1u);
  // unnormalised weighted latents [item][split][head][kv_rank], maximum and sum [item][split][head][2]
  const size_t out0 = ((size_t)item * splits + split) * ls.heads;
  if (scorer && sl == 0 && head0 + sh < ls.heads) {
    part_ml[(out0 + head0 + sh) * 2] = mx;
    part_ml[(out0 + head0 + sh) * 2 + 1] = sum;
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    const uint32_t d = (warp + 8 * m) * 16 + (lane >> 2);
    if (d >= ls.kv_rank) continue;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t h = head0 + n * 8 + (lane & 3) * 2 + (e & 1);
        if (h < ls.heads) part_o[(out0 + h) * ls.kv_rank + d + (e >> 1) * 8] = o[m][n][e];
      }
  }
}

// CTA (head and 64-wide tile of its values, tile of 16 listed rows): merged latents x W_uv, gated.
constexpr uint32_t kValueTile = 64, kValueRows = 16, kValueThreads = 256;
__global__ void __launch_bounds__(kValueThreads)
latent_value_kernel(const float *__restrict__ part_o, const float *__restrict__ part_ml, uint32_t ctx_splits, const bf16 *__restrict__ w_uv,
                    const float *__restrict__ gate, uint32_t splits, size_t split_stride, const uint32_t *__restrict__ row_list,
                    uint32_t rows, bf16 *__restrict__ out, uint32_t ldo, LatentShape ls) {
  extern __shared__ __align__(16) uint8_t smem[];
  const uint32_t pitch = ls.kv_rank * 2 + 16;
  uint8_t *w_s = smem, *o_s = smem + kValueTile * pitch;
  pdl_trigger();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t tiles = (ls.value_dim + kValueTile - 1) / kValueTile;
  const uint32_t head = blockIdx.x / tiles, v0 = (blockIdx.x % tiles) * kValueTile, row0 = blockIdx.y * kValueRows;
  const uint32_t nv = min(kValueTile, ls.value_dim - v0), n = min(kValueRows, rows - row0), groups = ls.kv_rank / 8;
  for (uint32_t i = tid; i < nv * groups; i += kValueThreads)
    cp_async16(w_s + (i / groups) * pitch + (i % groups) * 16, w_uv + ((size_t)head * ls.value_dim + v0 + i / groups) * ls.kv_rank + (i % groups) * 8);
  pdl_wait();
  // warp = 16 values (M) x 8 rows (N) of the product; its gate values are fetched before everything else
  const uint32_t vw = (warp & 3) * 16, rw = (warp >> 2) * 8;
  float g[4], c[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (uint32_t e = 0; e < 4; ++e) {
    const uint32_t r = rw + (lane & 3) * 2 + (e & 1), v = v0 + vw + (lane >> 2) + (e >> 1) * 8;
    g[e] = ls.gated && r < n && v < ls.value_dim
               ? fold(gate + (size_t)row_list[row0 + r] * ls.row_ld() + ls.q_cols() + ls.kv_cols() + head * ls.value_dim + v, splits, split_stride)
               : 0.f;
  }
  for (uint32_t r = warp; r < n; r += kValueThreads / 32) {  // one warp per row: lane s weighs split s, then all sum
    const size_t base = ((size_t)(row0 + r) * ctx_splits) * ls.heads + head;
    float2 ml = make_float2(-INFINITY, 0.f);
    if (lane < ctx_splits) ml = *reinterpret_cast<const float2 *>(part_ml + (base + (size_t)lane * ls.heads) * 2);
    const float mx = warp_max(ml.x), e = ml.x == -INFINITY ? 0.f : fast_exp2(ml.x - mx);
    const float wgt = e / warp_sum(e * ml.y);
    float4 a[4];  // kv_rank <= 512: four groups of four per lane, two splits of all of them in flight
#pragma unroll
    for (uint32_t k = 0; k < 4; ++k) a[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    for (uint32_t s0 = 0; s0 < ctx_splits; s0 += 2) {
      float4 x[2][4];
#pragma unroll
      for (uint32_t j = 0; j < 2; ++j)
#pragma unroll
        for (uint32_t k = 0; k < 4; ++k) {
          const uint32_t d = k * 128 + lane * 4;
          x[j][k] = s0 + j < ctx_splits && d < ls.kv_rank
                        ? *reinterpret_cast<const float4 *>(part_o + (base + (size_t)(s0 + j) * ls.heads) * ls.kv_rank + d)
                        : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
      for (uint32_t j = 0; j < 2; ++j) {
        const float w = __shfl_sync(0xffffffffu, wgt, (s0 + j) & 31u);
        if (s0 + j < ctx_splits) {
#pragma unroll
          for (uint32_t k = 0; k < 4; ++k) a[k].x += w * x[j][k].x, a[k].y += w * x[j][k].y, a[k].z += w * x[j][k].z, a[k].w += w * x[j][k].w;
        }
      }
    }
#pragma unroll
    for (uint32_t k = 0; k < 4; ++k)
      if (k * 128 + lane * 4 < ls.kv_rank) store4<bf16>(reinterpret_cast<bf16 *>(o_s + r * pitch) + k * 128 + lane * 4, a[k]);
  }
  cp_async_wait_all();
  __syncthreads();
  if (vw >= nv || rw >= n) return;  // rows beyond n stay undefined and are not stored
  const uint32_t mi = lane >> 3, rr = lane & 7;
  const uint32_t wa = smem_u32(w_s) + (vw + rr + (mi & 1) * 8) * pitch + (mi >> 1) * 16;
  const uint32_t ob = smem_u32(o_s) + (rw + rr) * pitch + mi * 16;
  for (uint32_t k = 0; k < ls.kv_rank; k += 32) {  // two steps of 16; the second may lie past the end
    uint32_t a[4], b[4];
    ldmatrix_x4(b, ob + k * 2);
    ldmatrix_x4(a, wa + k * 2);
    mma_bf16_16816(c, a, b[0], b[1]);
    if (k + 16 < ls.kv_rank) {
      ldmatrix_x4(a, wa + k * 2 + 32);
      mma_bf16_16816(c, a, b[2], b[3]);
    }
  }
#pragma unroll
  for (uint32_t e = 0; e < 4; ++e) {
    const uint32_t r = rw + (lane & 3) * 2 + (e & 1), v = v0 + vw + (lane >> 2) + (e >> 1) * 8;
    if (r < n && v < ls.value_dim)
      out[(size_t)row_list[row0 + r] * ldo + head * ls.value_dim + v] = __float2bfloat16_rn(ls.gated ? c[e] * sigmoid_f(g[e]) : c[e]);
  }
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

}  // namespace

template <typename T>
int launch_latent_prepare(const float *partial, uint32_t splits, size_t split_stride, const float *norm_w, const float *rope_cos,
                          const float *rope_sin, const uint32_t *positions, const uint32_t *slot_block, const uint32_t *slot_slot,
                          T *q, T *cache, LatentShape ls, uint32_t rows, cudaStream_t stream) {
  if (rows == 0) return ORION_OK;
  if (ls.dim % 4 == 0 && ls.rot_dim % 4 == 0 && ls.rope_dims % 4 == 0 && ls.kv_rank % 4 == 0 && ls.row_ld() % 4 == 0 &&
      ls.kv_cols() <= 4 * kPrepThreads) {
    const dim3 grid(rows, 1 + (ls.q_cols() / 4 + kPrepThreads - 1) / kPrepThreads);
    ORION_CUDA_CHECK("latent_prepare", launch_pdl(latent_prepare_vec_kernel<T>, grid, dim3(kPrepThreads), 0, stream, partial, splits,
                                                  split_stride, norm_w, rope_cos, rope_sin, positions, slot_block, slot_slot, q, cache, ls));
    return after_launch("latent_prepare");
  }
  ORION_CUDA_CHECK("latent_prepare", launch_pdl(latent_prepare_kernel<T>, dim3(rows), dim3(kPrepThreads), 0, stream, partial, splits,
                                                split_stride, norm_w, rope_cos, rope_sin, positions, slot_block, slot_slot, q, cache, ls));
  return after_launch("latent_prepare");
}

template <typename T>
int launch_latent_attention_generic(const T *q, const T *cache, const T *w_uk, const T *w_uv, const float *gate_partial,
                                    uint32_t splits, size_t split_stride, LatentShape ls, AttnBatch batch, T *out, uint32_t ldo,
                                    cudaStream_t stream) {
  if (batch.rows == 0) return ORION_OK;
  const size_t smem = (size_t)(ls.kv_cols() + ls.kv_rank + kGenKeys) * sizeof(float);
  if (smem > 200 * 1024) return set_error(ORION_ERR_INTERNAL, "latent size %u exceeds the attention kernel limit", ls.kv_rank);
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("latent_attention attr", ensure_dynamic_smem(latent_attention_generic_kernel<T>, 200 * 1024, attr_set));
  ORION_CUDA_CHECK("latent_attention", launch_pdl(latent_attention_generic_kernel<T>, dim3(batch.rows, ls.heads), dim3(kGenThreads), smem,
                                                  stream, q, cache, w_uk, w_uv, gate_partial, splits, split_stride, ls, batch, out, ldo));
  return after_launch("latent_attention");
}

bool latent_decode_supported(LatentShape ls) {
  return ls.kv_rank % 16 == 0 && ls.kv_rank <= 512 && ls.rot_dim % 16 == 0 && ls.dim % 16 == 0 && ls.dim > 0 && ls.dim <= 512 &&
         ls.kv_cols() <= 640 && ls.block_size == kCacheBlock && ls.row_stride % 16 == 8 && ls.row_stride >= ls.kv_cols();
}

namespace {
uint32_t decode_head_tiles(LatentShape ls) { return ls.heads <= 8 ? 1 : (ls.heads <= 16 ? 2 : 4); }
}  // namespace

uint32_t latent_decode_splits(LatentShape ls, uint32_t rows, uint32_t max_position) {
  const uint32_t nt = decode_head_tiles(ls), groups = (ls.heads + 8 * nt - 1) / (8 * nt);
  const uint32_t keys = ls.window ? std::min(ls.window, max_position + 1) : max_position + 1;
  const uint32_t tiles = (keys + kTileKeys - 1) / kTileKeys;
  // one resident wave of CTAs, as far as there are tiles to hand out
  const uint32_t resident = std::max(1u, std::min(8u, 227u * 1024u / (DecodeSmem(ls.row_stride, 8 * nt).total + 1024u)));
  const uint32_t want = 148 * resident / std::max(1u, rows * groups);
  return std::max(1u, std::min({want, tiles, kLatentMaxSplits}));
}

size_t latent_decode_scratch_floats(LatentShape ls, uint32_t rows, uint32_t splits) {
  return (size_t)rows * splits * ls.heads * (ls.kv_rank + 2);
}

int launch_latent_absorb(const bf16 *q, const bf16 *w_uk, const uint32_t *row_list, uint32_t rows, bf16 *qa, LatentShape ls,
                         cudaStream_t stream) {
  if (rows == 0) return ORION_OK;
  if (!latent_decode_supported(ls)) return set_error(ORION_ERR_INTERNAL, "latent decode attention does not cover this shape");
  const uint32_t tiles = (ls.kv_rank + kAbsorbTile - 1) / kAbsorbTile;
  const uint32_t smem = ls.dim * (kAbsorbTile * 2 + 16) + kRowTile * (ls.dim * 2 + 16);
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("latent_absorb attr", ensure_dynamic_smem(latent_absorb_kernel, 512 * (kAbsorbTile * 2 + 16) + kRowTile * (512 * 2 + 16), attr_set));
  ORION_CUDA_CHECK("latent_absorb", launch_pdl(latent_absorb_kernel, dim3(ls.heads * tiles, (rows + kRowTile - 1) / kRowTile), dim3(128), smem,
                                               stream, q, w_uk, row_list, rows, qa, ls));
  return after_launch("latent_absorb");
}

namespace {
template <int NT, int KQ, int MT>
int launch_decode(const bf16 *qa, const bf16 *cache, const uint32_t *row_list, const uint32_t *first_row, uint32_t rows, AttnBatch batch,
                  uint32_t splits, float *part_o, float *part_ml, LatentShape ls, cudaStream_t stream) {
  const DecodeSmem lay(ls.row_stride, 8 * NT);
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("latent_decode attr", ensure_dynamic_smem(latent_decode_kernel<NT, KQ, MT>, 227 * 1024, attr_set));
  ORION_CUDA_CHECK("latent_decode", launch_pdl(latent_decode_kernel<NT, KQ, MT>, dim3((ls.heads + 8 * NT - 1) / (8 * NT), rows, splits),
                                               dim3(kDecThreads), lay.total, stream, qa, cache, row_list, first_row, batch, splits, part_o,
                                               part_ml, ls));
  return after_launch("latent_decode");
}
template <int NT>
int launch_decode_nt(const bf16 *qa, const bf16 *cache, const uint32_t *row_list, const uint32_t *first_row, uint32_t rows, AttnBatch batch,
                     uint32_t splits, float *part_o, float *part_ml, LatentShape ls, cudaStream_t stream) {
  if (ls.kv_cols() <= 192) return launch_decode<NT, 3, 2>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream);
  if (ls.kv_cols() <= 384) return launch_decode<NT, 6, 3>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream);
  return launch_decode<NT, 10, 4>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream);
}
}  // namespace

int launch_latent_decode(const bf16 *qa, const bf16 *cache, const bf16 *w_uv, const float *gate_partial, uint32_t gate_splits,
                         size_t split_stride, const uint32_t *row_list, const uint32_t *first_row, uint32_t rows, AttnBatch batch,
                         uint32_t splits, float *scratch, LatentShape ls, bf16 *out, uint32_t ldo, cudaStream_t stream) {
  if (rows == 0) return ORION_OK;
  if (!latent_decode_supported(ls)) return set_error(ORION_ERR_INTERNAL, "latent decode attention does not cover this shape");
  float *part_o = scratch, *part_ml = scratch + (size_t)rows * splits * ls.heads * ls.kv_rank;
  switch (decode_head_tiles(ls)) {
    case 1: ORION_TRY(launch_decode_nt<1>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream)); break;
    case 2: ORION_TRY(launch_decode_nt<2>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream)); break;
    default: ORION_TRY(launch_decode_nt<4>(qa, cache, row_list, first_row, rows, batch, splits, part_o, part_ml, ls, stream)); break;
  }
  const uint32_t smem = (kValueTile + kValueRows) * (ls.kv_rank * 2 + 16) + 32;
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("latent_value attr", ensure_dynamic_smem(latent_value_kernel, (int)((kValueTile + kValueRows) * (512 * 2 + 16) + 32), attr_set));
  const dim3 grid(ls.heads * ((ls.value_dim + kValueTile - 1) / kValueTile), (rows + kValueRows - 1) / kValueRows);
  ORION_CUDA_CHECK("latent_value", launch_pdl(latent_value_kernel, grid, dim3(kValueThreads), smem, stream, part_o, part_ml, splits, w_uv, gate_partial,
                                              gate_splits, split_stride, row_list, rows, out, ldo, ls));
  return after_launch("latent_value");
}

int latent_poll_error(uint32_t *code) {
  uint32_t v = 0;
  ORION_CUDA_CHECK("latent attention error word", cudaMemcpyFromSymbol(&v, g_latent_error, sizeof v));
  if (v) {
    uint32_t zero = 0;
    ORION_CUDA_CHECK("latent attention error word", cudaMemcpyToSymbol(g_latent_error, &zero, sizeof zero));
  }
  *code = v;
  return ORION_OK;
}

#define ORION_INSTANTIATE(T)                                                                                                        \
  template int launch_latent_prepare<T>(const float *, uint32_t, size_t, const float *, const float *, const float *, const uint32_t *, \
                                        const uint32_t *, const uint32_t *, T *, T *, LatentShape, uint32_t, cudaStream_t);           \
  template int launch_latent_attention_generic<T>(const T *, const T *, const T *, const T *, const float *, uint32_t, size_t,        \
                                                  LatentShape, AttnBatch, T *, uint32_t, cudaStream_t);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
