// Latent attention over prompt portions on the 5th-generation tensor cores (bf16). For many query rows the keys and
// values are expanded once per token, K = W_uk c and V = W_uv c (one plain projection over the portion and the
// window before it), and attention runs on them per head: S = [Q_unrotated | Q_rotated] [K | shared rotated part]^T,
// O += P V, with S and O in tensor memory.
//   latent_gather_kernel      cached latents and rotated parts of each portion and the window before it, as rows
//   latent_prefill_tc_kernel  one CTA per (head, tile of 128 query rows of one sequence)
//     warp 0     one lane fetches K (the head's columns of the expanded rows, then the shared rotated part) and V of
//                64 keys by tiled TMA, 128-byte swizzled, one stage each
//     warp 1     allocates tensor memory; one lane issues the MMAs: S of the next tile goes into the other S
//                buffer while the softmax warps work on this one, then O (+)= P V (V is the MN-major operand)
//     warps 2-5  one thread per row: scores from tensor memory, masked by position and window, exponentials, P as bf16
//                into shared memory; O is rescaled in tensor memory only when a row's maximum moves by more than
//                2^8; at the end O / sum times the output gate
// Every wait is bounded; a wait that runs out sets the device error word and the CTA still frees its tensor memory.
#include "kernels.h"
#include "tcgen05.cuh"

#include <algorithm>
#include <map>
#include <mutex>
#include <tuple>

namespace orion {
namespace {

constexpr uint32_t kRows = kLatentTileRows, kKeys = 64, kThreads = 192;
constexpr uint32_t kQSlab = kRows * 128, kKSlab = kKeys * 128;  // 64 columns of the query tile / of a key tile
constexpr float kRescaleThreshold = 8.0f;                       // log2 units

__device__ uint32_t g_latent_prefill_error = 0;

__device__ __forceinline__ void softmax_bar() { asm volatile("bar.sync 1, 128;" ::: "memory"); }  // warps 2..5

// Shared memory in 64-column slabs: the unrotated and the rotated part of a query or key each start a slab.
struct PrefillSmem {
  uint32_t dim_slabs, slabs, value_slabs, k, v, p, bars, total;
  __host__ __device__ explicit PrefillSmem(const LatentShape &ls) {
    dim_slabs = (ls.dim + 63) / 64;
    slabs = dim_slabs + (ls.rot_dim + 63) / 64;
    value_slabs = (ls.value_dim + 63) / 64;
    k = slabs * kQSlab;
    v = k + slabs * kKSlab;
    p = v + value_slabs * kKSlab;
    bars = p + kRows * 128;
    total = bars + 128 + 1024;
  }
};
__host__ __device__ inline uint32_t tmem_columns(uint32_t value_dim) { return value_dim <= 128 ? 256 : 512; }
constexpr uint32_t kTmemO = 128;  // S: columns 0..63 and 64..127, O behind them

__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16 *__restrict__ cache, const uint32_t *__restrict__ tables_flat, const uint32_t *__restrict__ table_offsets,
                     const LatentPortion *__restrict__ portions, bf16 *__restrict__ latents, bf16 *__restrict__ rotated, LatentShape ls) {
  pdl_trigger();
  pdl_wait();
  const LatentPortion po = portions[blockIdx.y];
  const uint32_t i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= po.count) return;
  const uint32_t pos = po.position + i;
  const uint32_t *table = tables_flat + table_offsets[po.seq];
  const uint4 *src = reinterpret_cast<const uint4 *>(
      cache + ((size_t)table[pos / ls.block_size] * ls.block_size + pos % ls.block_size) * ls.row_stride);
  uint4 *lat = reinterpret_cast<uint4 *>(latents + (size_t)(po.row + i) * ls.kv_rank);
  uint4 *rot = reinterpret_cast<uint4 *>(rotated + (size_t)(po.row + i) * ls.rot_dim);
  const uint32_t n = ls.kv_rank / 8, all = ls.kv_cols() / 8;
  for (uint32_t g = lane; g < all; g += 32) {
    if (g < n) lat[g] = src[g];
    else rot[g - n] = src[g];
  }
}

__global__ void __launch_bounds__(kThreads)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_rot,
                         const __grid_constant__ CUtensorMap map_v, const bf16 *__restrict__ q, const float *__restrict__ gate,
                         uint32_t splits, size_t split_stride, const LatentTile *__restrict__ tiles, LatentShape ls,
                         bf16 *__restrict__ out, uint32_t ldo) {
  extern __shared__ uint8_t raw_smem[];
  uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(raw_smem) + 1023) & ~uintptr_t(1023));
  const PrefillSmem lay(ls);
  uint8_t *q_smem = smem, *k_smem = smem + lay.k, *v_smem = smem + lay.v, *p_smem = smem + lay.p;
  uint64_t *bars = reinterpret_cast<uint64_t *>(smem + lay.bars);
  uint64_t *k_full = bars, *k_empty = bars + 1, *v_full = bars + 2, *q_ready = bars + 3, *s_ready = bars + 4, *p_ready = bars + 6,
           *o_ready = bars + 7;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 8);
  __shared__ volatile uint32_t failed;

  const uint32_t head = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const LatentTile tile = tiles[blockIdx.y];
  const uint32_t first_key = ls.first_key(tile.position), last_key = tile.position + tile.num_rows - 1;
  const uint32_t ntiles = (last_key - first_key) / kKeys + 1;
  const uint32_t columns = tmem_columns(ls.value_dim);

  if (threadIdx.x == 0) {
    for (int i = 0; i < 8; ++i) mbar_init(&bars[i], 1);
    mbar_fence_init();
    failed = 0;
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, columns);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // only now: a dependent CTA that waits for this grid must not hold tensor memory that this CTA still needs
  pdl_trigger();
  const uint32_t tmem_base = *tmem_slot;
  bool ok = true;
  uint32_t k_issued = 0, v_issued = 0;  // copies of the producer lane
  // Once any wait of this CTA has run out, later waits give up at once: every thread still walks through the same
  // barriers, so nobody is left behind at a bar.sync.
  auto wait = [&](uint64_t *bar, uint32_t parity) -> bool {
    if (failed) return false;
    if (mbar_wait(bar, parity)) return true;
    failed = 1;
    return false;
  };

  if (warp == 0) {
    // ---- K/V producer ----
    if (lane == 0) {
      pdl_wait();
      const int row0 = tile.row_of_zero + (int)first_key;  // expanded row of the tile's first key
      const uint32_t k_bytes = lay.slabs * kKSlab, v_bytes = lay.value_slabs * kKSlab;
      for (uint32_t j = 0; j < ntiles; ++j) {
        const int row = row0 + (int)(j * kKeys);
        if (j > 0 && !wait(k_empty, (j - 1) & 1)) { ok = false; break; }
        mbar_arrive_expect_tx(k_full, k_bytes);
        ++k_issued;
        for (uint32_t h = 0; h < lay.dim_slabs; ++h) tma_load_3d(k_smem + h * kKSlab, &map_k, (int)(h * 64), (int)head, row, k_full);
        for (uint32_t h = lay.dim_slabs; h < lay.slabs; ++h)
          tma_load_2d(k_smem + h * kKSlab, &map_rot, (int)((h - lay.dim_slabs) * 64), row, k_full);
        if (j > 0 && !wait(o_ready, (j - 1) & 1)) { ok = false; break; }
        mbar_arrive_expect_tx(v_full, v_bytes);
        ++v_issued;
        for (uint32_t h = 0; h < lay.value_slabs; ++h) tma_load_3d(v_smem + h * kKSlab, &map_v, (int)(h * 64), (int)head, row, v_full);
      }
    }
  } else if (warp == 1) {
    // ---- MMA issue ----
    if (lane == 0) {
      const uint32_t idesc_s = idesc(kRows, kKeys, false), idesc_o = idesc(kRows, ls.value_dim, true);
      const uint32_t qa = smem_u32(q_smem), ka = smem_u32(k_smem), va = smem_u32(v_smem), pa = smem_u32(p_smem);
      auto scores = [&](uint32_t j) -> bool {
        if (!wait(k_full, j & 1)) return false;
        tc_fence_after();
        const uint32_t d = tmem_base + (j & 1) * kKeys;
        uint32_t fresh = 0;
        for (uint32_t ks = 0; ks < ls.dim / 16; ++ks, fresh = 1)
          umma_bf16(d, desc_k_sw128(qa + (ks >> 2) * kQSlab + (ks & 3) * 32), desc_k_sw128(ka + (ks >> 2) * kKSlab + (ks & 3) * 32), idesc_s, fresh);
        for (uint32_t ks = 0; ks < ls.rot_dim / 16; ++ks, fresh = 1) {
          const uint32_t h = lay.dim_slabs + (ks >> 2);
          umma_bf16(d, desc_k_sw128(qa + h * kQSlab + (ks & 3) * 32), desc_k_sw128(ka + h * kKSlab + (ks & 3) * 32), idesc_s, fresh);
        }
        umma_commit(&s_ready[j & 1]);
        umma_commit(k_empty);
        return true;
      };
      ok = wait(q_ready, 0) && scores(0);
      for (uint32_t j = 0; ok && j < ntiles; ++j) {
        if (j + 1 < ntiles && !scores(j + 1)) { ok = false; break; }
        if (!wait(p_ready, j & 1) || !wait(v_full, j & 1)) { ok = false; break; }
        tc_fence_after();
#pragma unroll
        for (uint32_t ks = 0; ks < kKeys / 16; ++ks)
          umma_bf16(tmem_base + kTmemO, desc_k_sw128(pa + ks * 32), desc_mn_sw128(va + ks * (16 * 128), kKSlab, 1024), idesc_o,
                    (j > 0 || ks > 0) ? 1u : 0u);
        umma_commit(o_ready);
      }
    }
  } else {
    // ---- softmax: thread = row ----
    const uint32_t quad = warp & 3;  // tensor-memory lanes this warp may touch
    const uint32_t m = quad * 32 + lane;
    const bool valid = m < tile.num_rows;
    const uint32_t row = tile.row_start + (valid ? m : 0);
    const int pos = valid ? (int)(tile.position + m) : -1, low = valid ? (int)ls.first_key((uint32_t)pos) : 0;
    const uint32_t taddr = tmem_base + ((quad * 32u) << 16);
    pdl_wait();
    {
      const uint4 *src = reinterpret_cast<const uint4 *>(q + (size_t)row * ls.q_cols() + (size_t)head * ls.q_dim());
      const uint32_t nd = ls.dim / 8, nr = ls.rot_dim / 8;
      for (uint32_t c = 0; c < nd + nr; ++c) {
        const uint4 v = valid ? src[c] : make_uint4(0u, 0u, 0u, 0u);
        const uint32_t g = c < nd ? c : lay.dim_slabs * 8 + (c - nd);  // 16-byte group in the slabbed row
        *reinterpret_cast<uint4 *>(q_smem + (g >> 3) * kQSlab + m * 128 + (((g & 7) ^ (m & 7)) << 4)) = v;
      }
    }
    fence_proxy_async_smem();
    softmax_bar();
    if (threadIdx.x == 64) mbar_arrive(q_ready);

    const float sl2 = ls.scale * 1.4426950408889634f;
    float ref = -INFINITY, l = 0.f;
    for (uint32_t j = 0; j < ntiles; ++j) {
      if (!__all_sync(0xffffffffu, wait(&s_ready[j & 1], (j >> 1) & 1))) ok = false;  // no break: the barriers below stay matched
      tc_fence_after();
      uint32_t sr[2][32];
      tmem_ld32(taddr + (j & 1) * kKeys, sr[0]);
      tmem_ld32(taddr + (j & 1) * kKeys + 32, sr[1]);
      tmem_ld_wait();
      const int key0 = (int)(first_key + j * kKeys);
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < (int)kKeys; ++i) {
        const float v = (key0 + i <= pos && key0 + i >= low) ? __uint_as_float(sr[i >> 5][i & 31]) * sl2 : -INFINITY;
        sr[i >> 5][i & 31] = __float_as_uint(v);
        mx = fmaxf(mx, v);
      }
      // The reference of the exponentials moves only when the maximum runs away from it.
      float corr = 1.0f;
      if (mx > ref + kRescaleThreshold || ref == -INFINITY) {
        const float nref = fmaxf(ref, mx);
        corr = (ref == -INFINITY) ? 1.0f : ex2(ref - nref);  // nothing accumulated yet under a reference of -inf
        ref = nref;
      }
      // P and O belong to the product of the previous tile until it has completed
      if (j > 0 && !__all_sync(0xffffffffu, wait(o_ready, (j - 1) & 1))) ok = false;
      tc_fence_after();
      if (__any_sync(0xffffffffu, corr != 1.0f) && j > 0) {
#pragma unroll 1
        for (uint32_t c = 0; c < ls.value_dim; c += 32) {  // columns past value_dim are this CTA's own and unused
          uint32_t orow[32];
          tmem_ld32(taddr + kTmemO + c, orow);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) orow[i] = __float_as_uint(__uint_as_float(orow[i]) * corr);
          tmem_st32(taddr + kTmemO + c, orow);
        }
        tmem_st_wait();
      }
      l *= corr;
      const float base = ref == -INFINITY ? 0.f : ref;
      uint8_t *p_row = p_smem + m * 128;
#pragma unroll
      for (int c = 0; c < (int)kKeys / 8; ++c) {
        float p[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          p[i] = ex2(__uint_as_float(sr[(c * 8 + i) >> 5][(c * 8 + i) & 31]) - base);
          l += p[i];
        }
        *reinterpret_cast<uint4 *>(p_row + ((c ^ (m & 7)) << 4)) =
            make_uint4(pack2(p[0], p[1]), pack2(p[2], p[3]), pack2(p[4], p[5]), pack2(p[6], p[7]));
      }
      tc_fence_before();         // the loads of S (and the rescale of O) precede the next MMAs
      fence_proxy_async_smem();  // P was written through the generic proxy, the MMA reads it through the async proxy
      softmax_bar();
      if (threadIdx.x == 64) mbar_arrive(p_ready);
    }
    // ---- epilogue: O / l, gated ----
    if (!__all_sync(0xffffffffu, wait(o_ready, (ntiles - 1) & 1))) ok = false;
    tc_fence_after();
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    bf16 *dst = out + (size_t)row * ldo + (size_t)head * ls.value_dim;
    const float *g = gate + (size_t)row * ls.row_ld() + ls.q_cols() + ls.kv_cols() + (size_t)head * ls.value_dim;
#pragma unroll 1
    for (uint32_t c = 0; c < ls.value_dim; c += 16) {
      uint32_t o[16];
      tmem_ld16(taddr + kTmemO + c, o);
      tmem_ld_wait();
      if (valid) {
        float r[16];
#pragma unroll
        for (uint32_t i = 0; i < 16; i += 4) {
          if (!ls.gated) {
#pragma unroll
            for (uint32_t k = 0; k < 4; ++k) r[i + k] = __uint_as_float(o[i + k]) * inv;
            continue;
          }
          const float4 gv = sum_slabs4(g + c + i, splits, split_stride);
          r[i] = __uint_as_float(o[i]) * inv * sigmoid_f(gv.x);
          r[i + 1] = __uint_as_float(o[i + 1]) * inv * sigmoid_f(gv.y);
          r[i + 2] = __uint_as_float(o[i + 2]) * inv * sigmoid_f(gv.z);
          r[i + 3] = __uint_as_float(o[i + 3]) * inv * sigmoid_f(gv.w);
        }
        *reinterpret_cast<uint4 *>(dst + c) = make_uint4(pack2(r[0], r[1]), pack2(r[2], r[3]), pack2(r[4], r[5]), pack2(r[6], r[7]));
        *reinterpret_cast<uint4 *>(dst + c + 8) = make_uint4(pack2(r[8], r[9]), pack2(r[10], r[11]), pack2(r[12], r[13]), pack2(r[14], r[15]));
      }
    }
  }
  if (!ok && lane == 0) atomicOr(&g_latent_prefill_error, 1u);
  tc_fence_before();
  __syncthreads();
  if (failed && threadIdx.x == 0) {  // nobody leaves while a copy may still land
    if (k_issued) mbar_wait(k_full, (k_issued - 1) & 1);
    if (v_issued) mbar_wait(v_full, (v_issued - 1) & 1);
  }
  if (warp == 1) tmem_dealloc(tmem_base, columns);
}

// ---- host side -----------------------------------------------------------------

// [rows][heads][cols] bf16 with `row_ld` elements between rows (heads = 1: a plain matrix); box of 64 columns x 64 rows.
int slab_map(const bf16 *base, uint32_t cols, uint32_t heads, uint32_t rows, uint32_t row_ld, bool by_head, const CUtensorMap **out) {
  static std::mutex mu;
  static std::map<std::tuple<const void *, uint32_t, uint32_t, uint32_t, uint32_t, bool>, CUtensorMap> cache;
  EncodeFn fn = encode_fn();
  if (!fn) return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: driver entry point missing");
  std::lock_guard<std::mutex> lock(mu);
  const auto key = std::make_tuple((const void *)base, cols, heads, rows, row_ld, by_head);
  auto it = cache.find(key);
  if (it == cache.end()) {
    if (cache.size() > 4096) cache.clear();
    CUtensorMap m;
    const cuuint64_t dims3[3] = {cols, heads, rows}, dims2[2] = {cols, rows};
    const cuuint64_t strides3[2] = {(cuuint64_t)cols * 2, (cuuint64_t)row_ld * 2}, strides2[1] = {(cuuint64_t)row_ld * 2};
    const cuuint32_t box3[3] = {64, 1, kKeys}, box2[2] = {64, kKeys}, ones[3] = {1, 1, 1};
    const CUresult r = fn(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, by_head ? 3 : 2, const_cast<bf16 *>(base), by_head ? dims3 : dims2,
                          by_head ? strides3 : strides2, by_head ? box3 : box2, ones, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS)
      return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: encode returned %d (%u columns, %u heads, %u rows)", (int)r,
                       cols, heads, rows);
    it = cache.emplace(key, m).first;
  }
  *out = &it->second;
  return ORION_OK;
}

}  // namespace

bool latent_prefill_supported(LatentShape ls) {
  return ls.dim > 0 && ls.dim % 16 == 0 && ls.rot_dim % 16 == 0 && ls.value_dim % 16 == 0 && ls.value_dim <= 256 && ls.kv_rank % 8 == 0 &&
         ls.kv_rank >= 64 && PrefillSmem(ls).total <= 226 * 1024 && encode_fn() != nullptr;
}

int launch_latent_gather(const bf16 *cache, const uint32_t *tables_flat, const uint32_t *table_offsets, const LatentPortion *portions,
                         uint32_t num_portions, uint32_t longest, bf16 *latents, bf16 *rotated, LatentShape ls, cudaStream_t stream) {
  if (num_portions == 0) return ORION_OK;
  ORION_CUDA_CHECK("latent_gather", launch_pdl(latent_gather_kernel, dim3((longest + 7) / 8, num_portions), dim3(256), 0, stream, cache,
                                               tables_flat, table_offsets, portions, latents, rotated, ls));
  count_launch();
  ORION_CUDA_CHECK("latent_gather", cudaGetLastError());
  return ORION_OK;
}

int launch_latent_prefill(const bf16 *q, const bf16 *expanded, const bf16 *rotated, uint32_t rows_capacity, const float *gate_partial,
                          uint32_t splits, size_t split_stride, const LatentTile *tiles, uint32_t num_tiles, LatentShape ls, bf16 *out,
                          uint32_t ldo, cudaStream_t stream) {
  if (num_tiles == 0) return ORION_OK;
  if (!latent_prefill_supported(ls)) return set_error(ORION_ERR_INTERNAL, "tensor-core latent attention does not cover this shape");
  const CUtensorMap *mk = nullptr, *mr = nullptr, *mv = nullptr;
  const uint32_t ld = ls.heads * (ls.dim + ls.value_dim);
  ORION_TRY(slab_map(expanded, ls.dim, ls.heads, rows_capacity, ld, true, &mk));
  ORION_TRY(slab_map(expanded + ls.heads * ls.dim, ls.value_dim, ls.heads, rows_capacity, ld, true, &mv));
  if (ls.rot_dim) ORION_TRY(slab_map(rotated, ls.rot_dim, 1, rows_capacity, ls.rot_dim, false, &mr));
  else mr = mk;
  // At least enough shared memory that the CTAs of an SM never ask for more tensor memory than it has (two of 256
  // columns, or one of 512 with no other kernel's CTA beside it).
  const uint32_t smem = std::max(PrefillSmem(ls).total, tmem_columns(ls.value_dim) == 256 ? 77u * 1024 : 132u * 1024);
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("latent_prefill attr", ensure_dynamic_smem(latent_prefill_tc_kernel, 226 * 1024, attr_set));
  ORION_CUDA_CHECK("latent_prefill", launch_pdl(latent_prefill_tc_kernel, dim3(ls.heads, num_tiles), dim3(kThreads), smem, stream, *mk, *mr,
                                                *mv, q, gate_partial, splits, split_stride, tiles, ls, out, ldo));
  count_launch();
  ORION_CUDA_CHECK("latent_prefill", cudaGetLastError());
  return ORION_OK;
}

int latent_prefill_poll_error(uint32_t *code) {
  uint32_t v = 0;
  ORION_CUDA_CHECK("latent prefill error word", cudaMemcpyFromSymbol(&v, g_latent_prefill_error, sizeof v));
  if (v) {
    uint32_t zero = 0;
    ORION_CUDA_CHECK("latent prefill error word", cudaMemcpyToSymbol(g_latent_prefill_error, &zero, sizeof zero));
  }
  *code = v;
  return ORION_OK;
}

}  // namespace orion
