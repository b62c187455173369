// Chunked-prefill paged attention on the 5th-generation tensor cores (bf16, head_dim 128, or 64 to 256
// with the FORM parameter; 16-token blocks): the same arithmetic as attention_prefill.cu (transformer.rs:281-326, causal by absolute
// position, attention.rs:252-253), with S = Q K^T and O += P V as tcgen05 MMAs whose accumulators
// live in tensor memory.
//
// One CTA per (kv head, tile of query rows of one sequence), two CTAs per SM. The MMA's M dimension
// is (query position, query head of the GQA group), 128 rows; a key tile is 64 keys = four KV blocks.
//   warp 0     one lane fetches K and V of a key tile with tiled TMA copies straight out of the paged
//              arena (3-D tensor maps over [chunk][slot][dim], one for K and one for V; a 16-slot x 64-dim box lands as
//              sixteen 128-byte rows, and because the arena keeps the 16-byte groups of a row XOR-permuted
//              by slot & 7, those rows ARE the 128-byte-swizzled operand layout the MMA expects);
//   warp 1     allocates tensor memory; one lane issues S = Q K^T (M 128, N 64, K 128) and, once the
//              softmax warps have written P, O (+)= P V (M 128, N 128, K 64; V is the MN-major operand; keys
//              that are values as well are one tile for both);
//   warps 2-5  one thread per row: read the row of S from tensor memory (lane = row, so max and sum
//              are thread-local), mask by position, exponentiate, write P as bf16 into the shared
//              memory the K tile has just vacated, and at the end scale O by 1 / sum and store it.
// O stays in tensor memory across key tiles. The running maximum a row's exponentials refer to is
// only moved when the true maximum exceeds it by more than 2^8; then the row's O is rescaled in
// tensor memory (load, multiply, store), which is rare after the first tiles.
// Every wait is bounded; a wait that runs out sets the device error word and the CTA still frees its
// tensor memory.
#include "kernels.h"
#include "tcgen05.cuh"

#include <cstdlib>
#include <map>
#include <mutex>
#include <tuple>

namespace orion {
namespace {

constexpr int kHd = 128, kBlk = 16;
constexpr int kM = 128;      // (position, head) rows per CTA
constexpr int kKeys = 64;    // keys per tile
constexpr int kThreads = 192;
// DK, DV: sizes of the K and V rows, multiples of 64. JOINT: one tile of rows is both K and V.
template <int DK, int DV, bool JOINT>
struct PrefillTcConfig {
  // Where tensor memory has room for it without costing a CTA, S has two buffers: the scores of the next key tile are computed under
  // the softmax of this one.
  static constexpr bool kTwoS = JOINT && DV == 128;
  static constexpr int kStages = kTwoS ? 3 : 2;
  static constexpr uint32_t kTmemO = kTwoS ? 128 : 64;  // S: the first columns of tensor memory, O behind them
  static constexpr int kQBytes = DK / 64 * kM * 128;     // 64-dim slabs of [128 rows][128 bytes]
  static constexpr int kKBytes = DK / 64 * kKeys * 128;  // 64-dim slabs of [64 keys][128 bytes]
  static constexpr int kVBytes = DV / 64 * kKeys * 128;
  static constexpr int kStageBytes = JOINT ? kKBytes : kKBytes + kVBytes;  // K tile, then V tile
  // P, [128 rows][128 bytes], takes the place of the K tile where that is large enough and not needed any more
  static constexpr bool kOwnP = JOINT || kKBytes < kM * 128;
  static constexpr int kPOffset = kQBytes + kStages * kStageBytes;
  static constexpr int kBarOffset = kPOffset + (kOwnP ? kM * 128 : 0);
  static constexpr int kFactorOffset = kBarOffset + 256;  // JOINT: the factors of a tile's keys, per stage
  static constexpr int kSmem = kFactorOffset + (JOINT ? kStages * kKeys * 4 : 0) + 1024;
  static constexpr uint32_t kTmemCols = DV <= 64 ? 128 : (DV <= 128 ? 256 : 512);
};
constexpr float kRescaleThreshold = 8.0f;    // log2 units

__device__ uint32_t g_prefill_tc_error = 0;

__device__ __forceinline__ void softmax_bar() { asm volatile("bar.sync 1, 128;" ::: "memory"); }  // warps 2..5

// FORM: 1 = the mask, sinks and gate of `form`, 2 = besides them the soft cap, the kept first positions and the gates of values; what
// is left out is compiled out. 3 = those of 1, one set of rows for keys and values with the factors of the keys
// (KvLayout::factor_elems), and the distance term.
template <int DK, int DV, int FORM>
__global__ void __launch_bounds__(kThreads, DV <= 128 ? 2 : 1)
paged_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v, const bf16 *__restrict__ q,
                        const bf16 *__restrict__ arena, KvLayout kv, uint32_t layer, AttnBatch batch, const PrefillTile *__restrict__ tiles,
                        uint32_t q_heads, bf16 *__restrict__ out, AttnForm form) {
  constexpr bool JOINT = FORM == 3;
  using Cfg = PrefillTcConfig<DK, DV, JOINT>;
  constexpr int kQBytes = Cfg::kQBytes, kKBytes = Cfg::kKBytes, kStageBytes = Cfg::kStageBytes, kStages = Cfg::kStages;
  constexpr uint32_t kTmemO = Cfg::kTmemO;
  constexpr bool kTwoS = Cfg::kTwoS;
  extern __shared__ uint8_t raw_smem[];
  uint8_t *smem = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(raw_smem) + 1023) & ~uintptr_t(1023));
  uint8_t *q_smem = smem;                 // [slab][row 128][128 B]
  uint8_t *ring = smem + kQBytes;         // [stage][K tile | V tile]
  float *factors = reinterpret_cast<float *>(smem + Cfg::kFactorOffset);  // [stage][key]
  auto p_tile = [&](uint32_t stage) { return Cfg::kOwnP ? smem + Cfg::kPOffset : ring + stage * kStageBytes; };
  uint64_t *kv_full = reinterpret_cast<uint64_t *>(smem + Cfg::kBarOffset);
  uint64_t *kv_empty = kv_full + kStages;
  uint64_t *q_ready = kv_empty + kStages;
  uint64_t *s_ready = q_ready + 1;
  uint64_t *p_ready = s_ready + 2;
  uint64_t *o_ready = p_ready + 1;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(o_ready + 1);

  if (!FORM) pdl_trigger();
  const uint32_t kvh = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const PrefillTile tile = tiles[blockIdx.y];
  const uint32_t group = q_heads / kv.num_kv_heads;
  const uint32_t *table = batch.tables_flat + batch.table_offsets[tile.seq];
  const uint32_t nblocks = tile.max_position / kBlk + 1;
  // key tiles start at the block of the first key that the tile's first row sees
  const uint32_t block0 = FORM ? form.range.first(batch.query_positions[tile.row_start]) / kBlk : 0;
  // before them come the blocks of the positions that every row keeps: index i -> logical block
  const uint32_t kept_blk = FORM == 2 ? form.range.kept_blocks(block0, kBlk) : 0;
  auto logical = [&](uint32_t i) { return FORM == 2 && i < kept_blk ? i : block0 - kept_blk + i; };
  const uint32_t ntiles = (kept_blk + nblocks - block0 + (kKeys / kBlk) - 1) / (kKeys / kBlk);

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&kv_full[s], 1);
      mbar_init(&kv_empty[s], 1);
    }
    mbar_init(q_ready, 1);
    mbar_init(&s_ready[0], 1);
    mbar_init(&s_ready[1], 1);
    mbar_init(p_ready, 1);
    mbar_init(o_ready, 1);
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // here only now: a dependent CTA that waits for this grid must not hold tensor memory that this CTA still needs
  if (FORM) pdl_trigger();
  const uint32_t tmem_base = *tmem_slot;
  bool ok = true;
  // Once any wait of this CTA has run out, later waits give up at once: every thread still walks
  // through the same barriers, so nobody is left behind at a bar.sync.
  __shared__ volatile uint32_t failed;
  if (threadIdx.x == 0) failed = 0;
  __syncthreads();
  auto wait = [&](uint64_t *bar, uint32_t parity) -> bool {
    if (failed) return false;
    if (mbar_wait(bar, parity)) return true;
    failed = 1;
    return false;
  };

  if (warp == 0) {
    // ---- K/V producer ----
    if (lane == 0) {
      pdl_wait();  // this step's K/V rows come from the preceding kernel
      const uint32_t chunk0 = layer * kv.num_blocks;
      for (uint32_t j = 0; j < ntiles; ++j) {
        const uint32_t s = j % kStages, use = j / kStages;
        if (!wait(&kv_empty[s], (use & 1) ^ 1)) { ok = false; break; }
        mbar_arrive_expect_tx(&kv_full[s], kStageBytes + (JOINT ? kKeys * 4 : 0));
        uint8_t *k_dst = ring + s * kStageBytes, *v_dst = k_dst + kKBytes;
#pragma unroll
        for (uint32_t b = 0; b < kKeys / kBlk; ++b) {
          // a block past the row's context repeats the first one: its keys are masked, its values must be finite
          const uint32_t lb = logical(j * (kKeys / kBlk) + b);
          const uint32_t block = table[lb < nblocks ? lb : block0];
          const int chunk = (int)((chunk0 + block) * kv.num_kv_heads + kvh);
#pragma unroll
          for (int h = 0; h < DK / 64; ++h)
            tma_load_3d(k_dst + h * (kKeys * 128) + b * (kBlk * 128), &map_k, h * 64, 0, chunk, &kv_full[s]);
          if (JOINT) {
            bulk_copy_g2s(factors + s * kKeys + b * kBlk, arena + kv.factor(layer, block, kvh, 0), kBlk * 4, &kv_full[s]);
            continue;
          }
#pragma unroll
          for (int h = 0; h < DV / 64; ++h)
            tma_load_3d(v_dst + h * (kKeys * 128) + b * (kBlk * 128), &map_v, h * 64, 0, chunk, &kv_full[s]);
        }
      }
    }
  } else if (warp == 1) {
    // ---- MMA issue ----
    if (lane == 0) {
      constexpr uint32_t idesc_s = idesc(kM, kKeys, false), idesc_o = idesc(kM, DV, true);
      const uint32_t qa = smem_u32(q_smem);
      // S = Q K^T: 64-dim slabs, four 16-dim steps each (+32 bytes inside the swizzle atom)
      auto scores = [&](uint32_t j) -> bool {
        const uint32_t s = j % kStages;
        if (!wait(&kv_full[s], (j / kStages) & 1)) return false;
        tc_fence_after();
        const uint32_t ka = smem_u32(ring + s * kStageBytes), b = kTwoS ? j & 1 : 0;
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks) {
          const uint32_t h = ks >> 2, kk = ks & 3;
          umma_bf16(tmem_base + b * kKeys, desc_k_sw128(qa + h * (kM * 128) + kk * 32), desc_k_sw128(ka + h * (kKeys * 128) + kk * 32),
                    idesc_s, ks > 0 ? 1u : 0u);
        }
        umma_commit(&s_ready[b]);
        return true;
      };
      if (!wait(q_ready, 0)) ok = false;
      if (kTwoS && ok && ntiles > 0) ok = scores(0);
      for (uint32_t j = 0; ok && j < ntiles; ++j) {
        const uint32_t s = j % kStages;
        // the other buffer's scores have been read: their P came before the product of the tile before
        if (kTwoS ? j + 1 < ntiles && !scores(j + 1) : !scores(j)) { ok = false; break; }
        const uint32_t ka = smem_u32(ring + s * kStageBytes), va = JOINT ? ka : ka + kKBytes;
        if (!wait(p_ready, j & 1)) { ok = false; break; }
        tc_fence_after();
        // O (+)= P V: P is [128 rows][64 keys] (where the K tile was, if it fits there); V is [key][dim]: MN-major, 16 keys per step
        const uint32_t pa = smem_u32(p_tile(s));
#pragma unroll
        for (int ks = 0; ks < kKeys / 16; ++ks)
          umma_bf16(tmem_base + kTmemO, desc_k_sw128(pa + ks * 32), desc_mn_sw128(va + ks * (16 * 128), kKeys * 128, 1024),
                    idesc_o, (j > 0 || ks > 0) ? 1u : 0u);
        umma_commit(o_ready);
        umma_commit(&kv_empty[s]);
      }
    }
  } else {
    // ---- softmax: thread = row ----
    const uint32_t quad = warp & 3;  // tensor-memory lanes this warp may touch
    const uint32_t m = quad * 32 + lane;
    const uint32_t pl = m / group;
    const bool valid = pl < tile.num_rows;
    const uint32_t row = tile.row_start + (valid ? pl : 0), head = kvh * group + m % group;
    const uint32_t taddr = tmem_base + ((quad * 32u) << 16);
    pdl_wait();  // q comes from the preceding kernel
    const int pos = valid ? (int)batch.query_positions[row] : -1;
    const int low = FORM && valid ? (int)form.range.first((uint32_t)pos) : 0;  // first key this row sees
    {
      const uint4 *src = reinterpret_cast<const uint4 *>(q + ((size_t)row * q_heads + head) * DK);
#pragma unroll
      for (uint32_t c = 0; c < DK / 8; ++c) {
        const uint4 v = valid ? src[c] : make_uint4(0u, 0u, 0u, 0u);
        *reinterpret_cast<uint4 *>(q_smem + (c >> 3) * (kM * 128) + m * 128 + (((c & 7) ^ (m & 7)) << 4)) = v;
      }
    }
    fence_proxy_async_smem();
    softmax_bar();
    if (threadIdx.x == 64) mbar_arrive(q_ready);

    float sl2 = FORM && form.scale != 0.f ? form.scale * 1.4426950408889634f : 1.4426950408889634f / sqrtf((float)DK);
    const int keep = FORM == 2 ? (int)form.range.keep : 0;
    // A soft cap leaves scores in the log2 domain. Where every score of a warp's tile is at most kTaylor of the cap it is a polynomial, and
    // unless the cap is very high the exponentials need no running maximum.
    constexpr float kTaylor = 0.35f;
    float cap_in = 0.f, cap_out = 0.f, small = 0.f, taylor[5] = {};
    bool fixed = false;
    if (FORM == 2 && form.softcap != 0.f) {
      const float y = (form.scale != 0.f ? form.scale : 1.0f / sqrtf((float)DK)) / form.softcap;  // tanh's argument per unit of q.k
      cap_out = form.softcap * 1.4426950408889634f, cap_in = 2.f * 1.4426950408889634f * y;
      small = kTaylor / y;
      // tanh(x) = x - x^3 / 3 + 2 x^5 / 15 - 17 x^7 / 315 + 62 x^9 / 2835 - ...
      taylor[0] = cap_out * y, taylor[1] = taylor[0] * y * y * (-1.f / 3.f), taylor[2] = taylor[0] * y * y * y * y * (2.f / 15.f);
      taylor[3] = taylor[2] * y * y * (-17.f / 42.f), taylor[4] = taylor[3] * y * y * (-62.f / 153.f);
      sl2 = 1.f;
      fixed = cap_out <= 60.f && !form.sinks;
    }
    float dist_mult = 0.f, dist_rate = 0.f;
    if (JOINT && form.dist_mult) dist_mult = form.dist_mult[head], dist_rate = form.dist_rate[head];
    float ref = -INFINITY, l = 0.f;
    if (FORM && form.sinks) ref = form.sinks[head] * 1.4426950408889634f, l = 1.f;
    for (uint32_t j = 0; j < ntiles; ++j) {
      const uint32_t s = j % kStages;
      const uint32_t sb = kTwoS ? j & 1 : 0;
      if (!__all_sync(0xffffffffu, wait(&s_ready[sb], (kTwoS ? j >> 1 : j) & 1))) ok = false;  // no break: the barriers below stay matched
      tc_fence_after();
      uint32_t sr[2][32];
      tmem_ld32(taddr + sb * kKeys, sr[0]);
      tmem_ld32(taddr + sb * kKeys + 32, sr[1]);
      tmem_ld_wait();
      const bool straight = FORM != 2 || j * (kKeys / kBlk) >= kept_blk || kept_blk == block0;  // the tile's keys follow one another
      const int key0 = (int)(logical(j * (kKeys / kBlk)) * kBlk);
      float mx = -INFINITY;
      if (JOINT) {
        if (!__all_sync(0xffffffffu, wait(&kv_full[s], (j / kStages) & 1))) ok = false;  // the factors landed with the tile
        const float4 *factor = reinterpret_cast<const float4 *>(factors + s * kKeys);
        // The distance term at key i is dist_mult log2(mid + dist_rate t), t = 31.5 - i. Where t is small beside mid / dist_rate for every
        // row of the warp, it is a polynomial in t: log(1 + x) = x - x^2 / 2 + x^3 / 3 - ... up to x^5 for |x| below 1/8, with
        // t a constant of each key and the even and odd powers shared by the keys t and -t.
        const float mid = fmaf(dist_rate, (float)(pos - key0) - 31.5f, 1.f), x1 = __fdividef(dist_rate, mid);
        if (__all_sync(0xffffffffu, !valid || (mid > 0.f && x1 <= 0.125f / 31.5f))) {
          const float lead = dist_mult * 1.4426950408889634f, x2 = x1 * x1;
          const float c0 = dist_mult * fast_log2(mid), c1 = lead * x1, c2 = lead * x2 * -0.5f, c3 = lead * x2 * x1 * (1.f / 3.f),
                      c4 = lead * x2 * x2 * -0.25f, c5 = lead * x2 * x2 * x1 * 0.2f;
#pragma unroll
          for (int i = 0; i < kKeys / 2; i += 4) {
            const float4 f = factor[i / 4], g = factor[kKeys / 4 - 1 - i / 4];
            const float fs[4] = {f.x, f.y, f.z, f.w}, gs[4] = {g.w, g.z, g.y, g.x};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const int a = i + k, b = kKeys - 1 - a;
              const float t = 31.5f - (float)a, t2 = t * t;
              const float even = fmaf(fmaf(c4, t2, c2), t2, c0), odd = fmaf(fmaf(c5, t2, c3), t2, c1);
              sr[a >> 5][a & 31] = __float_as_uint(fmaf(__uint_as_float(sr[a >> 5][a & 31]), fs[k] * sl2, -fmaf(odd, t, even)));
              sr[b >> 5][b & 31] = __float_as_uint(fmaf(__uint_as_float(sr[b >> 5][b & 31]), gs[k] * sl2, fmaf(odd, t, -even)));
            }
          }
        } else {
          const float near = fmaf(dist_rate, (float)(pos - key0), 1.f);  // the logarithm's argument at the tile's first key
#pragma unroll
          for (int i = 0; i < kKeys; i += 4) {
            const float4 f = factor[i / 4];
            const float fs[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const float v = __uint_as_float(sr[(i + k) >> 5][(i + k) & 31]) * (fs[k] * sl2);
              sr[(i + k) >> 5][(i + k) & 31] = __float_as_uint(v - dist_mult * fast_log2(fmaf(-dist_rate, (float)(i + k), near)));
            }
          }
        }
      }
      if (FORM == 2 && form.softcap != 0.f) {
        float most = 0.f;
#pragma unroll
        for (int i = 0; i < kKeys; ++i) most = fmaxf(most, fabsf(__uint_as_float(sr[i >> 5][i & 31])));
        if (__all_sync(0xffffffffu, most <= small)) {
#pragma unroll
          for (int i = 0; i < kKeys; ++i) {
            const float x = __uint_as_float(sr[i >> 5][i & 31]), x2 = x * x;
            sr[i >> 5][i & 31] = __float_as_uint(x * fmaf(x2, fmaf(x2, fmaf(x2, fmaf(x2, taylor[4], taylor[3]), taylor[2]), taylor[1]), taylor[0]));
          }
        } else {
#pragma unroll
          for (int i = 0; i < kKeys; ++i) sr[i >> 5][i & 31] = __float_as_uint(softcap_log2(__uint_as_float(sr[i >> 5][i & 31]), cap_in, cap_out));
        }
      }
      // most key tiles are seen whole by every row of a warp (rows past the tile are not stored)
      if (straight && __all_sync(0xffffffffu, !valid || (key0 + kKeys - 1 <= pos && (!FORM || key0 >= low)))) {
        if (FORM == 2 && fixed) {
          mx = 0.f;
        } else {
#pragma unroll
          for (int i = 0; i < kKeys; ++i) {
            const float v = JOINT ? __uint_as_float(sr[i >> 5][i & 31]) : __uint_as_float(sr[i >> 5][i & 31]) * sl2;
            sr[i >> 5][i & 31] = __float_as_uint(v);
            mx = fmaxf(mx, v);
          }
        }
      } else {
        int from[kKeys / kBlk];  // first key of every block
#pragma unroll
        for (int b = 0; b < kKeys / kBlk; ++b) from[b] = straight ? key0 + b * kBlk : (int)(logical(j * (kKeys / kBlk) + b) * kBlk);
#pragma unroll
        for (int i = 0; i < kKeys; ++i) {
          const int key = from[i / kBlk] + i % kBlk;
          const float v = (key <= pos && (!FORM || key >= low || (FORM == 2 && key < keep))) ? __uint_as_float(sr[i >> 5][i & 31]) * (JOINT ? 1.f : sl2) : -INFINITY;
          sr[i >> 5][i & 31] = __float_as_uint(v);
          mx = fmaxf(mx, v);
        }
      }
      if (FORM == 2 && fixed) mx = 0.f;  // the reference stays at zero: the exponents are between plus and minus the cap
      // The reference of the exponentials moves only when the maximum runs away from it.
      float corr = 1.0f;
      if (mx > ref + kRescaleThreshold || ref == -INFINITY) {
        const float nref = fmaxf(ref, mx);
        corr = (ref == -INFINITY) ? 1.0f : ex2(ref - nref);  // nothing accumulated yet under a reference of -inf
        ref = nref;
      }
      if (kTwoS && j > 0) {  // P and O belong to the product of the previous tile until it has completed
        if (!__all_sync(0xffffffffu, wait(o_ready, (j - 1) & 1))) ok = false;
        tc_fence_after();
      }
      if (__any_sync(0xffffffffu, corr != 1.0f) && j > 0) {
        // rescale this warp's rows of O in tensor memory (the MMAs of the previous tile have completed:
        // with one buffer S of this tile was issued after them)
#pragma unroll 1
        for (uint32_t c = 0; c < DV; c += 32) {
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
      uint8_t *p_row = p_tile(s) + m * 128;
#pragma unroll
      for (int c = 0; c < kKeys / 8; ++c) {
        float p[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          p[i] = ex2(__uint_as_float(sr[(c * 8 + i) >> 5][(c * 8 + i) & 31]) - base);
          l += p[i];
        }
        *reinterpret_cast<uint4 *>(p_row + ((c ^ (m & 7)) << 4)) =
            make_uint4(pack2(p[0], p[1]), pack2(p[2], p[3]), pack2(p[4], p[5]), pack2(p[6], p[7]));
      }
      tc_fence_before();        // the loads of S (and the rescale of O) precede the next MMAs
      fence_proxy_async_smem();  // P was written through the generic proxy, the MMA reads it through the async proxy
      softmax_bar();
      if (threadIdx.x == 64) mbar_arrive(p_ready);
    }
    // ---- epilogue: O / l ----
    if (!__all_sync(0xffffffffu, ntiles == 0 || wait(o_ready, (ntiles - 1) & 1))) ok = false;
    tc_fence_after();
    float inv = l > 0.f ? 1.0f / l : 0.f;
    if (FORM && form.gate) inv *= form.gate[(size_t)row * q_heads + head];
    const uint32_t od = FORM && form.out_dim ? form.out_dim : DV, ldo = FORM && form.ldo ? form.ldo : q_heads * od;
    const bool whole_groups = !FORM || (od % 8 == 0 && ldo % 8 == 0);
    bf16 *dst = out + (size_t)row * ldo + (size_t)head * od;
    const bf16 *vgate = FORM == 2 && form.value_gate ? static_cast<const bf16 *>(form.value_gate) + ((size_t)row * q_heads + head) * od : nullptr;
#pragma unroll 1
    for (uint32_t c = 0; c < DV; c += 32) {
      uint32_t orow[32];
      tmem_ld32(taddr + kTmemO + c, orow);
      tmem_ld_wait();
      if (FORM == 2 && vgate && valid) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          if (c + i >= od) continue;
          if (whole_groups) {
            const uint4 g = *reinterpret_cast<const uint4 *>(vgate + c + i);
            const uint32_t w[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int k = 0; k < 8; ++k)  // the bits of a bf16 are the upper half of the f32
              orow[i + k] = __float_as_uint(__uint_as_float(orow[i + k]) * __uint_as_float(k & 1 ? w[k / 2] & 0xFFFF0000u : w[k / 2] << 16));
          } else {
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (c + i + k < od) orow[i + k] = __float_as_uint(__uint_as_float(orow[i + k]) * __bfloat162float(vgate[c + i + k]));
          }
        }
      }
      if (valid) {
#pragma unroll
        for (int i = 0; i < 32; i += 8) {
          if (!whole_groups) {
#pragma unroll
            for (int k = 0; k < 8; ++k)
              if (c + i + k < od) dst[c + i + k] = __float2bfloat16_rn(__uint_as_float(orow[i + k]) * inv);
          } else if (!FORM || c + i < od) {
            *reinterpret_cast<uint4 *>(dst + c + i) =
                make_uint4(pack2(__uint_as_float(orow[i]) * inv, __uint_as_float(orow[i + 1]) * inv),
                           pack2(__uint_as_float(orow[i + 2]) * inv, __uint_as_float(orow[i + 3]) * inv),
                           pack2(__uint_as_float(orow[i + 4]) * inv, __uint_as_float(orow[i + 5]) * inv),
                           pack2(__uint_as_float(orow[i + 6]) * inv, __uint_as_float(orow[i + 7]) * inv));
          }
        }
      }
    }
  }
  if (!ok && lane == 0) atomicOr(&g_prefill_tc_error, 1u);
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, Cfg::kTmemCols);
}

// ---- host side -----------------------------------------------------------------

// The K or the V rows of the arena as [chunk = (layer, block, kv head)][16 slots][dims]; a box is 16 rows x 64 dims with
// no swizzle of its own (the rows are stored pre-permuted).
int arena_map(const bf16 *arena, KvLayout kv, bool values, const CUtensorMap **out) {
  static std::mutex mu;
  static std::map<std::tuple<const void *, uint64_t, uint32_t, uint64_t, bool>, CUtensorMap> cache;
  EncodeFn fn = encode_fn();
  if (!fn) return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: driver entry point missing");
  const uint64_t chunks = (uint64_t)kv.num_layers * kv.num_blocks * kv.num_kv_heads;
  std::lock_guard<std::mutex> lock(mu);
  auto key = std::make_tuple((const void *)arena, chunks, kv.head_dim, (uint64_t)kv.chunk_elems(), values);
  auto it = cache.find(key);
  if (it == cache.end()) {
    if (cache.size() > 4096) cache.clear();
    CUtensorMap m;
    const cuuint64_t cols = values ? kv.v_dim() : kv.head_dim;
    const cuuint64_t dims[3] = {cols, (cuuint64_t)kBlk, chunks};
    const cuuint64_t strides[2] = {cols * 2, (cuuint64_t)kv.chunk_elems() * 2};
    bf16 *base = const_cast<bf16 *>(arena) + (values && !kv.factor_elems ? (size_t)kBlk * kv.head_dim : 0);
    const cuuint32_t box[3] = {64, (cuuint32_t)kBlk, 1};
    const cuuint32_t estr[3] = {1, 1, 1};
    const CUresult r = fn(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, base, dims, strides, box, estr,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                          CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS)
      return set_error(ORION_ERR_BACKEND, "backend cuda failed at tensor map: encode returned %d (arena of %llu chunks)", (int)r,
                       (unsigned long long)chunks);
    it = cache.emplace(key, m).first;
  }
  *out = &it->second;
  return ORION_OK;
}

template <int DK, int DV, int FORM>
int launch_prefill_tc(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer, AttnBatch batch, const PrefillTile *tiles,
                      uint32_t num_tiles, uint32_t q_heads, AttnForm form, bf16 *out, cudaStream_t stream) {
  using Cfg = PrefillTcConfig<DK, DV, FORM == 3>;
  const CUtensorMap *mk = nullptr, *mv = nullptr;
  ORION_TRY(arena_map(arena, kv, false, &mk));
  ORION_TRY(arena_map(arena, kv, true, &mv));
  static bool attr_set[kMaxDeviceOrdinals] = {};
  ORION_CUDA_CHECK("paged_prefill_tc attr", ensure_dynamic_smem(paged_prefill_tc_kernel<DK, DV, FORM>, Cfg::kSmem, attr_set));
  ORION_CUDA_CHECK("paged_prefill_tc", launch_pdl(paged_prefill_tc_kernel<DK, DV, FORM>, dim3(kv.num_kv_heads, num_tiles), dim3(kThreads),
                                                  (size_t)Cfg::kSmem, stream, *mk, *mv, q, arena, kv, layer, batch, tiles, q_heads, out, form));
  count_launch();
  ORION_CUDA_CHECK("paged_prefill_tc", cudaGetLastError());
  return ORION_OK;
}

// Tuning A/B and the parity tests of both paths: ORION_PREFILL_TC=0 keeps the mma.sync kernel.
bool g_prefill_tc = std::getenv("ORION_PREFILL_TC") ? std::atoi(std::getenv("ORION_PREFILL_TC")) != 0 : true;

}  // namespace

bool prefill_attention_tc_supported(KvLayout kv, uint32_t q_heads, const void *arena) {
  return g_prefill_tc && prefill_attention_supported(kv, q_heads) && (reinterpret_cast<uintptr_t>(arena) & 15) == 0 &&
         (uint64_t)kv.num_layers * kv.num_blocks * kv.num_kv_heads < (1ull << 31) && encode_fn() != nullptr;
}

int launch_paged_attention_prefill_tc(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer, AttnBatch batch,
                                      const PrefillTile *tiles, uint32_t num_tiles, uint32_t q_heads, bf16 *out,
                                      cudaStream_t stream) {
  if (num_tiles == 0) return ORION_OK;
  if (!prefill_attention_tc_supported(kv, q_heads, arena))
    return set_error(ORION_ERR_INTERNAL, "tensor-core prefill attention does not cover this shape");
  return launch_prefill_tc<kHd, kHd, 0>(q, arena, kv, layer, batch, tiles, num_tiles, q_heads, AttnForm{}, out, stream);
}

int launch_paged_attention_prefill_form(const bf16 *q, const bf16 *arena, KvLayout kv, uint32_t layer, AttnBatch batch,
                                        const PrefillTile *tiles, uint32_t num_tiles, uint32_t q_heads, AttnForm form, bf16 *out,
                                        cudaStream_t stream) {
  if (num_tiles == 0) return ORION_OK;
  if (!attention_form_supported(kv, q_heads) || encode_fn() == nullptr)
    return set_error(ORION_ERR_INTERNAL, "tensor-core prefill attention does not cover this shape");
  const uint32_t dk = kv.head_dim, dv = kv.v_dim();
  if (form.dist_mult && !kv.factor_elems) return set_error(ORION_ERR_INTERNAL, "prefill attention takes distance terms where keys and values are one");
  if (kv.factor_elems) {
    if (form.softcap != 0.f || form.range.keep || form.value_gate)
      return set_error(ORION_ERR_INTERNAL, "prefill attention over one set of rows has no soft cap, kept positions or gates of values");
    auto joint = dk == 256 ? launch_prefill_tc<256, 256, 3> : (dk == 64 ? launch_prefill_tc<64, 64, 3> : launch_prefill_tc<128, 128, 3>);
    return joint(q, arena, kv, layer, batch, tiles, num_tiles, q_heads, form, out, stream);
  }
  auto pick = [&](auto plain, auto more) { return form.softcap != 0.f || form.range.keep || form.value_gate ? more : plain; };
  auto run = dk == 256  ? pick(launch_prefill_tc<256, 256, 1>, launch_prefill_tc<256, 256, 2>)
             : dk == 64 ? (dv == 64 ? pick(launch_prefill_tc<64, 64, 1>, launch_prefill_tc<64, 64, 2>)
                                    : pick(launch_prefill_tc<64, 128, 1>, launch_prefill_tc<64, 128, 2>))
                        : (dv == 64 ? pick(launch_prefill_tc<128, 64, 1>, launch_prefill_tc<128, 64, 2>)
                                    : pick(launch_prefill_tc<128, 128, 1>, launch_prefill_tc<128, 128, 2>));
  return run(q, arena, kv, layer, batch, tiles, num_tiles, q_heads, form, out, stream);
}

int prefill_tc_poll_error(uint32_t *code) {
  uint32_t v = 0;
  ORION_CUDA_CHECK("prefill error word", cudaMemcpyFromSymbol(&v, g_prefill_tc_error, sizeof v));
  if (v) {
    uint32_t zero = 0;
    ORION_CUDA_CHECK("prefill error word", cudaMemcpyToSymbol(g_prefill_tc_error, &zero, sizeof zero));
  }
  *code = v;
  return ORION_OK;
}

}  // namespace orion
