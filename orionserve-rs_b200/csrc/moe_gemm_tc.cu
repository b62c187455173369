// Grouped products of a mixture of experts on the 5th-generation tensor cores (bf16): the projection kernel of gemm_tc.cu over
// a list of tiles, each a run of rows that share one expert. As there, the weight matrix is the M operand (128 rows per
// MMA) and the rows are N, so an expert's weights are streamed once per tile, whatever the number of its rows; a tile's rows
// past its count belong to the next expert and are not stored.
//   CTA (x: weight tiles; y: row tile, the shared expert's first; z: k split), 256 threads
//   warp 0     one lane streams the expert's weights by TMA, 64-wide k slabs, 128-byte swizzled (the shared expert's before the
//              preceding kernel has ended; the others once the tile list is there)
//   warp 2     one lane does the same with the tile's rows
//   warp 1     allocates tensor memory, one lane issues the MMAs
//   warps 4-7  epilogue (all eight warps where an activation is computed): f32 rows, or f(w g) * (w u), f a gated activation, of neighbouring gate and up rows with the row's score w, or
//              an activation f(w u) without a gate
// Every wait is bounded; a wait that runs out sets the device error word and the CTA still frees its tensor memory.
#include "kernels.h"
#include "tcgen05.cuh"

#include <algorithm>
#include <map>
#include <mutex>
#include <tuple>

namespace orion {
namespace {

constexpr uint32_t kTileN = 128, kSlabK = 64, kThreads = 256;

__device__ uint32_t g_moe_error = 0;

// WST / XST: stages of the weight and the row ring; MT: weight tiles per CTA.
template <int TOKN, int WST, int XST, int MT>
struct MoeConfig {
  static constexpr int kWBytes = MT * kTileN * kSlabK * 2, kXBytes = TOKN * kSlabK * 2;
  static constexpr int kXOffset = WST * kWBytes, kBarOffset = kXOffset + XST * kXBytes;
  static constexpr int kSmemBytes = kBarOffset + 1024 + 256;
  static constexpr uint32_t kTmemCols = MT * TOKN < 32 ? 32 : MT * TOKN;
  static_assert(kTmemCols <= 512 && (kTmemCols & (kTmemCols - 1)) == 0 && kSmemBytes <= 232448, "tile does not fit an SM");
};

struct TcArgs {
  uint32_t n, k, shared_n, shared_k, shared_tiles, rows, sorted_rows, splits;
  const MoeTile *tiles;
  const float *row_score;
  bf16 *act, *shared_act;
  float *out, *shared_out;
  GatedAct f, shared_f;
};

// GATED: 0 = f32 products, 1 = SwiGLU, 2 = the gated activations of the arguments, 3 = no gate, the exact GELU of every product.
template <int TOKN, int WST, int XST, int MT, int GATED>
__global__ void __launch_bounds__(kThreads)
moe_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const __grid_constant__ CUtensorMap map_sw,
                   const __grid_constant__ CUtensorMap map_sx, TcArgs a) {
  using Cfg = MoeConfig<TOKN, WST, XST, MT>;
  extern __shared__ uint8_t raw_smem[];
  uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(raw_smem) + 1023) & ~uintptr_t(1023));
  uint8_t *w_ring = smem, *x_ring = smem + Cfg::kXOffset;
  uint64_t *full_w = reinterpret_cast<uint64_t *>(smem + Cfg::kBarOffset), *empty_w = full_w + WST, *full_x = empty_w + WST, *empty_x = full_x + XST,
           *acc_ready = empty_x + XST;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(acc_ready + 1);
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool shared = blockIdx.y < a.shared_tiles;
  const uint32_t n = shared ? a.shared_n : a.n, k = shared ? a.shared_k : a.k, n0 = blockIdx.x * (MT * kTileN), split = blockIdx.z;
  if (n0 >= n) return;  // the grid is as wide as the wider of the two products
  if (threadIdx.x == 0) {
    for (int s = 0; s < WST; ++s) mbar_init(&full_w[s], 1), mbar_init(&empty_w[s], 1);
    for (int s = 0; s < XST; ++s) mbar_init(&full_x[s], 1), mbar_init(&empty_x[s], 1);
    mbar_init(acc_ready, 1);
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // only now: a dependent CTA that waits for this grid must not hold tensor memory that this CTA still needs
  pdl_trigger();
  const uint32_t tmem_base = *tmem_slot;

  MoeTile tile;
  if (shared) {
    tile = MoeTile{0, blockIdx.y * TOKN, min((uint32_t)TOKN, a.rows - blockIdx.y * TOKN)};
  } else {
    pdl_wait();
    tile = a.tiles[blockIdx.y - a.shared_tiles];
  }
  const bool live = tile.count > 0;
  const uint32_t nkb = (k + kSlabK - 1) / kSlabK;
  const uint32_t kb_begin = split * nkb / a.splits, my_kb = live ? (split + 1) * nkb / a.splits - kb_begin : 0;
  const CUtensorMap *mw = shared ? &map_sw : &map_w, *mx = shared ? &map_sx : &map_x;
  bool ok = true;

  if (warp == 0) {
    if (lane == 0) {
      for (uint32_t i = 0; i < my_kb; ++i) {
        const uint32_t s = i % WST;
        if (!mbar_wait(&empty_w[s], ((i / WST) & 1) ^ 1)) { ok = false; break; }
        mbar_arrive_expect_tx(&full_w[s], Cfg::kWBytes);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)  // rows past the matrix read as zeros, rows past the expert belong to the next one
          tma_load_2d(w_ring + s * Cfg::kWBytes + mt * (kTileN * kSlabK * 2), mw, (int)((kb_begin + i) * kSlabK),
                      (int)(tile.expert * n + n0 + mt * kTileN), &full_w[s]);
      }
    }
  } else if (warp == 2) {
    if (lane == 0) {
      pdl_wait();
      for (uint32_t i = 0; i < my_kb; ++i) {
        const uint32_t s = i % XST;
        if (!mbar_wait(&empty_x[s], ((i / XST) & 1) ^ 1)) { ok = false; break; }
        mbar_arrive_expect_tx(&full_x[s], Cfg::kXBytes);
        tma_load_2d(x_ring + s * Cfg::kXBytes, mx, (int)((kb_begin + i) * kSlabK), (int)tile.row, &full_x[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && my_kb > 0) {
      constexpr uint32_t id = idesc(kTileN, TOKN, false);
      for (uint32_t i = 0; i < my_kb; ++i) {
        const uint32_t sw = i % WST, sx = i % XST;
        if (!mbar_wait(&full_w[sw], (i / WST) & 1) || !mbar_wait(&full_x[sx], (i / XST) & 1)) { ok = false; break; }
        tc_fence_after();
        const uint32_t wt = smem_u32(w_ring + sw * Cfg::kWBytes), xt = smem_u32(x_ring + sx * Cfg::kXBytes);
#pragma unroll
        for (uint32_t kk = 0; kk < kSlabK / 16; ++kk)
#pragma unroll
          for (int mt = 0; mt < MT; ++mt)
            umma_bf16(tmem_base + mt * TOKN, desc_k_sw128(wt + mt * (kTileN * kSlabK * 2) + kk * 32), desc_k_sw128(xt + kk * 32), id, (i > 0 || kk > 0) ? 1u : 0u);
        umma_commit(&empty_w[sw]);
        umma_commit(&empty_x[sx]);
      }
      umma_commit(acc_ready);
    }
  }
  __syncwarp();
  // The epilogue is on all eight warps where it computes something: the four that may read the same rows of tensor memory share the
  // chunks of a tile with the four others. Values come before the tests for rows past the end, so that they overlap.
  constexpr uint32_t kGroups = GATED ? 2 : 1;
  if (live && (kGroups == 2 || warp >= 4)) {
    const uint32_t lq = warp & 3;
    pdl_wait();  // the results may still be read by the kernel before, and the scores come from one
    if (my_kb > 0 && !mbar_wait(acc_ready, 0)) ok = false;
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    float *out = shared ? a.shared_out + (size_t)split * a.rows * n : a.out + (size_t)split * a.sorted_rows * n;
    bf16 *act = shared ? a.shared_act : a.act;
    constexpr int kBatch = TOKN >= 64 ? (GATED ? 2 : 4) : (GATED ? 1 : TOKN / 16);
#pragma unroll 1
    for (int mb = kGroups == 2 && warp < 4 ? 16 * kBatch : 0; mb < MT * TOKN; mb += 16 * kBatch * kGroups) {
      uint32_t rr[kBatch][16];
      if (ok && my_kb > 0) {
#pragma unroll
        for (int b = 0; b < kBatch; ++b) tmem_ld16(tmem_base + ((lq * 32u) << 16) + (uint32_t)(mb + 16 * b), rr[b]);
        tmem_ld_wait();
      } else {
#pragma unroll
        for (int b = 0; b < kBatch; ++b)
#pragma unroll
          for (int j = 0; j < 16; ++j) rr[b][j] = 0u;
      }
#pragma unroll
      for (int b = 0; b < kBatch; ++b) {
        const int mc = mb + 16 * b;
        const uint32_t c = mc % TOKN, nn = n0 + (mc / TOKN) * kTileN + lq * 32 + lane;  // first row of the tile in this chunk, weight row
        if (c >= tile.count) continue;  // warp-uniform
        if (GATED == 3) {
          bf16 v[16], *to = act + (size_t)(tile.row + c) * n + nn;
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const float w = shared || !a.row_score ? 1.f : a.row_score[tile.row + min(c + j, tile.count - 1)];
            v[j] = __float2bfloat16_rn(gelu_erf<bf16>(w * __uint_as_float(rr[b][j])));
          }
          if (nn < n) {
#pragma unroll
            for (int j = 0; j < 16; ++j, to += n)
              if (c + j < tile.count) *to = v[j];
          }
        } else if (GATED) {
          // lane 2i holds gate f, lane 2i + 1 up f, of the same f for these 16 rows; a pair trades halves and each
          // finishes one row of every two
          const uint32_t odd = lane & 1u, f = nn >> 1, ffn = n >> 1;
          bf16 v[8], *to = act + (size_t)(tile.row + c + odd) * ffn + f;
#pragma unroll
          for (int jj = 0; jj < 8; ++jj) {
            const uint32_t send = odd ? rr[b][2 * jj] : rr[b][2 * jj + 1];
            const uint32_t recv = __shfl_xor_sync(0xffffffffu, send, 1);
            const float w = shared || !a.row_score ? 1.f : a.row_score[tile.row + min(c + 2 * jj + odd, tile.count - 1)];
            const float g = w * __uint_as_float(odd ? recv : rr[b][2 * jj]), u = w * __uint_as_float(odd ? rr[b][2 * jj + 1] : recv);
            v[jj] = __float2bfloat16_rn(GATED == 1 ? silu_for<bf16>(g) * u : gated<bf16>(shared ? a.shared_f : a.f, g, u));
          }
          if (nn < n) {
#pragma unroll
            for (int jj = 0; jj < 8; ++jj, to += 2 * (size_t)ffn)
              if (c + 2 * jj + odd < tile.count) *to = v[jj];
          }
        } else if (nn < n) {
#pragma unroll
          for (int j = 0; j < 16; ++j)
            if (c + j < tile.count) out[(size_t)(tile.row + c + j) * n + nn] = __uint_as_float(rr[b][j]);
        }
      }
    }
  }
  if (!ok && lane == 0) atomicOr(&g_moe_error, 1u);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, Cfg::kTmemCols);
}

// [rows][k] bf16, box of 64 k x box_rows, 128-byte swizzle.
int matrix_map(const bf16 *base, uint64_t rows, uint64_t k, uint32_t box_rows, const CUtensorMap **out) {
  static std::mutex mu;
  static std::map<std::tuple<const void *, uint64_t, uint64_t, uint32_t>, CUtensorMap> cache;
  EncodeFn fn = encode_fn();
  if (!fn) return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: driver entry point missing");
  std::lock_guard<std::mutex> lock(mu);
  const auto key = std::make_tuple((const void *)base, rows, k, box_rows);
  auto it = cache.find(key);
  if (it == cache.end()) {
    CUtensorMap m;
    const cuuint64_t dims[2] = {k, rows}, strides[1] = {k * 2};
    const cuuint32_t box[2] = {kSlabK, box_rows}, ones[2] = {1, 1};
    const CUresult r = fn(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<bf16 *>(base), dims, strides, box, ones, CU_TENSOR_MAP_INTERLEAVE_NONE,
                          CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS)
      return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: encode returned %d (rows %llu k %llu)", (int)r, (unsigned long long)rows,
                       (unsigned long long)k);
    it = cache.emplace(key, m).first;
  }
  *out = &it->second;
  return ORION_OK;
}

template <int TOKN, int WST, int XST, int MT>
int launch_product(const MoeProduct &p, bool swiglu, uint32_t splits, MoePlan plan, cudaStream_t stream) {
  using Cfg = MoeConfig<TOKN, WST, XST, MT>;
  const CUtensorMap *mw, *mx, *msw, *msx;
  ORION_TRY(matrix_map(p.w, (uint64_t)p.experts * p.n, p.k, kTileN, &mw));
  ORION_TRY(matrix_map(p.x, p.sorted_rows, p.k, TOKN, &mx));
  msw = mw, msx = mx;
  if (p.shared_n) {
    ORION_TRY(matrix_map(p.shared_w, p.shared_n, p.shared_k, kTileN, &msw));
    ORION_TRY(matrix_map(p.shared_x, p.rows, p.shared_k, TOKN, &msx));
  }
  const uint32_t shared_tiles = p.shared_n ? (p.rows + TOKN - 1) / TOKN : 0;
  const TcArgs a{p.n, p.k, p.shared_n, p.shared_k, shared_tiles, p.rows, p.sorted_rows, splits, p.tiles, p.row_score, p.act, p.shared_act, p.out, p.shared_out, p.f, p.shared_f};
  const dim3 grid((std::max(p.n, p.shared_n) + MT * kTileN - 1) / (MT * kTileN), shared_tiles + plan.tiles, splits);
  static bool attr_set[4][kMaxDeviceOrdinals] = {};
  const int form = !swiglu ? 0 : (p.f.plain() ? 3 : (p.f.kind == kGatedSilu && p.shared_f.kind == kGatedSilu ? 1 : 2));
  auto kernel = form == 0   ? moe_gemm_tc_kernel<TOKN, WST, XST, MT, 0>
                : form == 1 ? moe_gemm_tc_kernel<TOKN, WST, XST, MT, 1>
                : form == 2 ? moe_gemm_tc_kernel<TOKN, WST, XST, MT, 2>
                            : moe_gemm_tc_kernel<TOKN, WST, XST, MT, 3>;
  ORION_CUDA_CHECK("moe_gemm attr", ensure_dynamic_smem(kernel, Cfg::kSmemBytes, attr_set[form]));
  ORION_CUDA_CHECK("moe_gemm", launch_pdl(kernel, grid, dim3(kThreads), (size_t)Cfg::kSmemBytes, stream, *mw, *mx, *msw, *msx, a));
  count_launch();
  ORION_CUDA_CHECK("moe_gemm", cudaGetLastError());
  return ORION_OK;
}

}  // namespace

bool moe_tc_supported(MoeShape s) {
  auto fits = [](uint32_t k) { return k >= kSlabK && k % 8 == 0; };
  return fits(s.hidden) && fits(s.ffn) && (s.shared_ffn == 0 || fits(s.shared_ffn)) && encode_fn() != nullptr;
}

int launch_moe_product_tc(const MoeProduct &p, bool swiglu, uint32_t splits, MoePlan plan, cudaStream_t stream) {
  if (swiglu && splits != 1) return set_error(ORION_ERR_INTERNAL, "the fused SwiGLU epilogue needs one k split");
  switch (plan.tile_rows) {
    case 16: return launch_product<16, 6, 3, 1>(p, swiglu, splits, plan, stream);
    case 32: return launch_product<32, 6, 3, 1>(p, swiglu, splits, plan, stream);
    case 64: return launch_product<64, 5, 3, 1>(p, swiglu, splits, plan, stream);
    case 128: return launch_product<128, 4, 2, 1>(p, swiglu, splits, plan, stream);
    default: return launch_product<256, 3, 3, 2>(p, swiglu, splits, plan, stream);
  }
}

int moe_poll_error(uint32_t *code) {
  uint32_t v = 0;
  ORION_CUDA_CHECK("mixture error word", cudaMemcpyFromSymbol(&v, g_moe_error, sizeof v));
  if (v) {
    uint32_t zero = 0;
    ORION_CUDA_CHECK("mixture error word", cudaMemcpyToSymbol(g_moe_error, &zero, sizeof zero));
  }
  *code = v;
  return ORION_OK;
}

}  // namespace orion
