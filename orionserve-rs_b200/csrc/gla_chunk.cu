// Gated linear attention over prompt portions, 64 rows ("a chunk") at a time. With b_i the sum of the logarithms of the decays of
// a chunk's rows up to i (one value per key channel) and S the state before the chunk,
//   o_i = (q_i e^(b_i)) S + sum_(j <= i) A_ij v_j,   A_ij = sum_d q_id k_jd e^(b_id - b_jd)
//   S  <- e^(b_63) S + sum_j (k_j e^(b_63 - b_j)) v_j^T
// and every exponential is of something that is not positive.
//   gla_prepare_kernel  CTA per (head, chunk), all chunks at once: decays and their sums, A, and the two scaled operands in bf16
//   gla_scan_kernel     CTA per (head, 32 value columns, sequence), chunk after chunk: S stays in registers as f32 accumulators of
//                       mma.sync and is read by the products with q as two bf16 parts (value and remainder)
//   gla_finish_kernel   warp per (row, head): norm over the head, gate
// The exponents of A's operands are relative to the start of the 16 rows of i, so that only the factor of j inside those 16 rows can
// exceed one; where a channel decays by more than 2^60 within 16 rows, those 16 x 16 pairs are summed one by one instead.
#include "gla.cuh"
#include "mma.cuh"

#include <algorithm>

namespace orion {
namespace {

constexpr uint32_t kC = kGlaChunk, kThreads = 256, kWarps = kThreads / 32, kSub = 16, kSubs = kC / kSub;
constexpr uint32_t kSlice = 32;                           // value columns per CTA of the scan
constexpr uint32_t kVStride = kSlice + 8, kAStride = kC + 8;  // rows of an odd number of 16-byte groups: fragments load without conflicts
constexpr size_t kPrepareSmem = 226 * 1024;
constexpr float kMostDecay = -60.f;                       // log2, of 16 rows

__device__ uint32_t g_gla_error = 0;

// One (chunk, head) of the scratch buffer: q and k [64][row], A [64][kAStride], the chunk's whole decay [dims] in f32, and the values as
// slices [64][kVStride].
struct ItemLayout {
  uint32_t dims, row, slices, k, a, decay, v, bytes;
  __host__ __device__ explicit ItemLayout(const GlaShape &s) {
    dims = (s.dim + 15) / 16 * 16, row = dims + 8, slices = (s.value_dim + kSlice - 1) / kSlice;
    k = kC * row * 2, a = 2 * k, decay = a + kC * kAStride * 2, v = decay + dims * 4, bytes = v + slices * slice_bytes();
  }
  static __host__ __device__ constexpr uint32_t slice_bytes() { return kC * kVStride * 2; }
};
// Row stride of f32 rows whose float2 fragments (8 rows x 4 pairs) fall into different banks.
__host__ __device__ inline uint32_t float_stride(uint32_t dims) { return dims % 32 ? dims + 24 : dims + 8; }

constexpr uint32_t kRankStride = kC + 4;
inline size_t prepare_smem(const GlaShape &s) {
  const ItemLayout L(s);
  return (3 * (size_t)kC * float_stride(L.dims) + kSubs * L.dims + (size_t)kRankStride * s.rank) * sizeof(float);
}

// x and y as bf16, and what that leaves out.
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}

// VEC: four columns at once, from at most SLABS slabs (0: any number).
template <bool VEC, int SLABS>
__device__ __forceinline__ float4 load_quad(const float *p, uint32_t splits, size_t stride, uint32_t valid) {
  if constexpr (VEC) {
    return valid ? sum_slabs4_most<SLABS>(p, splits, stride) : make_float4(0.f, 0.f, 0.f, 0.f);
  } else {
    float v[4];
#pragma unroll
    for (uint32_t i = 0; i < 4; ++i) v[i] = i < valid ? fold_slabs(p + i, splits, stride) : 0.f;
    return make_float4(v[0], v[1], v[2], v[3]);
  }
}
__device__ __forceinline__ float4 exp2_4(float4 x) { return make_float4(fast_exp2(x.x), fast_exp2(x.y), fast_exp2(x.z), fast_exp2(x.w)); }
__device__ __forceinline__ uint2 pack_product4(float4 a, float4 b) { return make_uint2(pack_bf16x2(a.x * b.x, a.y * b.y), pack_bf16x2(a.z * b.z, a.w * b.w)); }

template <bool VEC, int SLABS>
__global__ void __launch_bounds__(kThreads, 3)
gla_prepare_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<bf16> w,
                   const GlaChunk *__restrict__ chunks, uint8_t *__restrict__ items) {
  extern __shared__ __align__(16) float smem[];
  __shared__ uint32_t steep;  // bit I: rows 16 I .. 16 I + 15 decay by more than the limit in some channel
  const ItemLayout L(s);
  const uint32_t SD = float_stride(L.dims), tid = threadIdx.x, head = blockIdx.x;
  float *q = smem, *k = q + kC * SD, *b = k + kC * SD, *total = b + kC * SD, *a1 = total + kSubs * L.dims;  // a1 [rank][kRankStride]
  uint8_t *item = items + ((size_t)blockIdx.y * s.heads + head) * L.bytes;
  pdl_trigger();
  if (tid == 0) steep = 0;
  const GlaChunk ch = chunks[blockIdx.y];
  pdl_wait();
  const uint32_t nq = s.q_cols(), nv = s.v_cols(), quads = L.dims / 4, vquads = L.slices * kSlice / 4;
  const float *p = partial + (size_t)ch.row * s.ld;
  const float qs = 1.0f / sqrtf((float)s.dim);
  for (uint32_t i = tid; i < kC * s.rank; i += kThreads) {
    const uint32_t t = i / s.rank, r = i % s.rank;
    const float *src = p + (size_t)t * s.ld + 2 * nq + 2 * nv + r;
    a1[r * kRankStride + t] = t < ch.count ? (SLABS == 1 ? *src : fold_slabs(src, splits, split_stride)) : 0.f;
  }
#pragma unroll 4
  for (uint32_t i = tid; i < kC * quads; i += kThreads) {
    const uint32_t t = i / quads, d = i % quads * 4, valid = t < ch.count && d < s.dim ? s.dim - d : 0;
    const float *src = p + (size_t)t * s.ld + head * s.dim + d;
    const float4 x = load_quad<VEC, SLABS>(src, splits, split_stride, valid), y = load_quad<VEC, SLABS>(src + nq, splits, split_stride, valid);
    *reinterpret_cast<float4 *>(q + t * SD + d) = make_float4(x.x * qs, x.y * qs, x.z * qs, x.w * qs);
    *reinterpret_cast<float4 *>(k + t * SD + d) = y;
  }
#pragma unroll 4
  for (uint32_t i = tid; i < kC * vquads; i += kThreads) {
    const uint32_t t = i / vquads, v = i % vquads * 4, valid = t < ch.count && v < s.value_dim ? s.value_dim - v : 0;
    const float4 x = load_quad<VEC, SLABS>(p + (size_t)t * s.ld + 2 * nq + head * s.value_dim + v, splits, split_stride, valid);
    bf16 *dst = reinterpret_cast<bf16 *>(item + L.v + v / kSlice * ItemLayout::slice_bytes()) + t * kVStride + v % kSlice;
    *reinterpret_cast<uint2 *>(dst) = make_uint2(pack_bf16x2(x.x, x.y), pack_bf16x2(x.z, x.w));
  }
  __syncthreads();

  // Logarithms (base 2) of the decays, summed within 16 rows, then over the chunk.
  for (uint32_t i = tid; i < kSubs * L.dims; i += kThreads) {
    const uint32_t d = i % L.dims, sub = i / L.dims;
    float z[kSub];
    const bool live = d < s.dim;
    const size_t c = (size_t)head * s.dim + (live ? d : 0);
    const float bias = w.bias[c], unit = 1.4426950408889634f / s.tau;
#pragma unroll
    for (uint32_t t = 0; t < kSub; ++t) z[t] = bias;
#pragma unroll 4
    for (uint32_t r = 0; r < s.rank; ++r) {
      const float wr = __bfloat162float(w.decay[c * s.rank + r]);
      const float4 *a = reinterpret_cast<const float4 *>(a1 + r * kRankStride + sub * kSub);
#pragma unroll
      for (uint32_t t = 0; t < kSub; t += 4) {
        const float4 x = a[t / 4];
        z[t] = fmaf(wr, x.x, z[t]), z[t + 1] = fmaf(wr, x.y, z[t + 1]), z[t + 2] = fmaf(wr, x.z, z[t + 2]), z[t + 3] = fmaf(wr, x.w, z[t + 3]);
      }
    }
    float sum = 0.f;
#pragma unroll
    for (uint32_t t = 0; t < kSub; ++t) {
      if (live && sub * kSub + t < ch.count) sum += log_sigmoid_fast(z[t]) * unit;
      b[(sub * kSub + t) * SD + d] = sum;
    }
    total[i] = sum;
    if (!(sum > kMostDecay)) atomicOr(&steep, 1u << sub);
  }
  __syncthreads();
  for (uint32_t i = L.dims + tid; i < kSubs * L.dims; i += kThreads) {
    const uint32_t d = i % L.dims, sub = i / L.dims;
    float before = 0.f;
    for (uint32_t u = 0; u < sub; ++u) before += total[u * L.dims + d];
#pragma unroll
    for (uint32_t t = 0; t < kSub; ++t) b[(sub * kSub + t) * SD + d] += before;
  }
  __syncthreads();

  // The operands of the scan.
  const float *last = b + (kC - 1) * SD;
#pragma unroll 2
  for (uint32_t i = tid; i < kC * quads; i += kThreads) {
    const uint32_t t = i / quads, d = i % quads * 4;
    const float4 x = *reinterpret_cast<const float4 *>(q + t * SD + d), y = *reinterpret_cast<const float4 *>(k + t * SD + d);
    const float4 at = *reinterpret_cast<const float4 *>(b + t * SD + d), e = *reinterpret_cast<const float4 *>(last + d);
    bf16 *dst = reinterpret_cast<bf16 *>(item) + t * L.row + d;
    *reinterpret_cast<uint2 *>(dst) = pack_product4(x, exp2_4(at));
    *reinterpret_cast<uint2 *>(dst + L.k / 2) = pack_product4(y, exp2_4(make_float4(e.x - at.x, e.y - at.y, e.z - at.z, e.w - at.w)));
  }
  for (uint32_t d = tid; d < L.dims; d += kThreads) reinterpret_cast<float *>(item + L.decay)[d] = fast_exp2(last[d]);

  // A in blocks of 16 x 16, on and below the diagonal (nothing reads the others): a warp takes one or two of a row of blocks.
  const uint32_t lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2, warp = tid >> 5;
  constexpr uint32_t kPlan[kWarps] = {0x302, 0x322, 0x202, 0x221, 0x101, 0x111, 0x001, 0};  // I, first J, number of J
  uint32_t plan = 0;
#pragma unroll
  for (uint32_t i = 0; i < kWarps; ++i)
    if (warp == i) plan = kPlan[i];
  const uint32_t I = plan >> 8, J0 = plan >> 4 & 15, nJ = plan & 15, i0 = I * kSub;
  if (nJ == 0) return;
  bf16 *A = reinterpret_cast<bf16 *>(item + L.a);
  const float *ref = I > 0 ? b + (i0 - 1) * SD : nullptr;
  auto pair = [&](const float *x, uint32_t row, uint32_t d, float sign, float2 r) {
    const float2 v = *reinterpret_cast<const float2 *>(x + row * SD + d), at = *reinterpret_cast<const float2 *>(b + row * SD + d);
    return pack_bf16x2(v.x * fast_exp2(sign * (at.x - r.x)), v.y * fast_exp2(sign * (at.y - r.y)));
  };
  float acc[2][2][4] = {};
  const bool slow = steep >> I & 1u;
  for (uint32_t d0 = 0; d0 < L.dims; d0 += 16) {
    uint32_t a[4];
    float2 r[2];
#pragma unroll
    for (uint32_t h = 0; h < 2; ++h) {
      const uint32_t d = d0 + h * 8 + t2;
      r[h] = ref ? *reinterpret_cast<const float2 *>(ref + d) : make_float2(0.f, 0.f);
      a[2 * h] = pair(q, i0 + g, d, 1.f, r[h]);
      a[2 * h + 1] = pair(q, i0 + g + 8, d, 1.f, r[h]);
    }
#pragma unroll
    for (uint32_t n = 0; n < 2; ++n) {
      if (n >= nJ || (slow && J0 + n == I)) continue;
#pragma unroll
      for (uint32_t nt = 0; nt < 2; ++nt) {
        uint32_t bk[2];
#pragma unroll
        for (uint32_t h = 0; h < 2; ++h) bk[h] = pair(k, (J0 + n) * kSub + nt * 8 + g, d0 + h * 8 + t2, -1.f, r[h]);
        mma_bf16_16816(acc[n][nt], a, bk[0], bk[1]);
      }
    }
  }
#pragma unroll
  for (uint32_t n = 0; n < 2; ++n) {
    if (n >= nJ) continue;
    const uint32_t j0 = (J0 + n) * kSub;
    if (slow && J0 + n == I) {
#pragma unroll
      for (uint32_t e = 0; e < 8; ++e) {
        const uint32_t i = i0 + g + (e & 2 ? 8 : 0), j = j0 + (e >> 2) * 8 + t2 + (e & 1);
        float sum = 0.f;
        if (j <= i)
          for (uint32_t d = 0; d < s.dim; ++d) sum += q[i * SD + d] * k[j * SD + d] * fast_exp2(b[i * SD + d] - b[j * SD + d]);
        acc[n][e >> 2][e & 3] = sum;
      }
    }
#pragma unroll
    for (uint32_t nt = 0; nt < 2; ++nt)
#pragma unroll
      for (uint32_t h = 0; h < 2; ++h) {
        const uint32_t i = i0 + g + 8 * h, j = j0 + nt * 8 + t2;
        const float x = j <= i ? acc[n][nt][2 * h] : 0.f, y = j + 1 <= i ? acc[n][nt][2 * h + 1] : 0.f;
        *reinterpret_cast<uint32_t *>(A + i * kAStride + j) = pack_bf16x2(x, y);
      }
  }
}

// What the scan holds in shared memory: a ring of (operands of a chunk, one slice of its values), the state in two bf16 parts (two copies
// where they fit, so that one barrier per chunk is enough), barriers.
struct ScanPlan {
  uint32_t stages = 0, copies = 0, smem = 0;
  explicit ScanPlan(const GlaShape &s) {
    const ItemLayout L(s);
    const uint32_t stage = L.v + ItemLayout::slice_bytes(), parts = 2 * L.dims * kVStride * 2;
    for (uint32_t budget : {113u * 1024, 227u * 1024})  // two CTAs per SM if that can be
      for (uint32_t c = 2; c >= 1; --c)
        for (uint32_t n = 3; n >= 2; --n)
          if (smem == 0 && n * stage + c * parts + 64 <= budget) stages = n, copies = c, smem = n * stage + c * parts + 64;
  }
};

// DT: tiles of 16 key channels per warp.
template <int DT>
__global__ void __launch_bounds__(kThreads)
gla_scan_kernel(const uint8_t *__restrict__ items, GlaShape s, float *__restrict__ state, StateBatch sb, const GlaChunk *__restrict__ chunks,
                const GlaPortion *__restrict__ portions, float *__restrict__ o_out, uint32_t stages, uint32_t copies) {
  extern __shared__ __align__(128) uint8_t ring[];
  const ItemLayout L(s);
  const uint32_t stage_bytes = L.v + ItemLayout::slice_bytes(), part = L.dims * kVStride;  // elements of one part of the state
  bf16 *parts = reinterpret_cast<bf16 *>(ring + stages * stage_bytes);
  uint64_t *full = reinterpret_cast<uint64_t *>(ring + stages * stage_bytes + copies * 4 * part);
  const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t2 = (lane & 3) * 2;
  const uint32_t head = blockIdx.x / L.slices, slice = blockIdx.x % L.slices, v0 = slice * kSlice;
  pdl_trigger();
  const GlaPortion por = portions[blockIdx.y];
  if (tid < stages) mbar_init(&full[tid], 1);
  mbar_fence_init();
  const size_t base = (size_t)head * s.dim * s.value_dim;
  const uint32_t rd = sb.read[por.seq];

  // S[d][v] as accumulators: tile dt of this warp covers channels 16 (warp + 8 dt) ..., four tiles of 8 columns.
  float S[DT][4][4];
  auto each = [&](auto &&f) {  // f(value, channel, column)
#pragma unroll
    for (int dt = 0; dt < DT; ++dt)
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) f(S[dt][nt][e], (warp + kWarps * dt) * 16 + g + (e & 2 ? 8 : 0), v0 + nt * 8 + t2 + (e & 1));
  };
  each([&](float &x, uint32_t d, uint32_t v) {
    x = rd != kNoState && d < s.dim && v < s.value_dim ? state[rd * s.state_floats() + base + (size_t)d * s.value_dim + v] : 0.f;
  });
  auto publish = [&](uint32_t copy) {  // the state as value and remainder
    bf16 *hi = parts + copy * 2 * part, *lo = hi + part;
#pragma unroll
    for (int dt = 0; dt < DT; ++dt) {
      const uint32_t d = (warp + kWarps * dt) * 16 + g;
      if (d >= L.dims) continue;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          uint32_t a, b;
          split2(S[dt][nt][2 * h], S[dt][nt][2 * h + 1], a, b);
          const uint32_t at = (d + 8 * h) * kVStride + nt * 8 + t2;
          *reinterpret_cast<uint32_t *>(hi + at) = a;
          *reinterpret_cast<uint32_t *>(lo + at) = b;
        }
    }
  };
  publish(0);
  __syncthreads();
  pdl_wait();
  auto issue = [&](uint32_t c) {  // one thread
    const uint8_t *src = items + ((size_t)(por.chunk + c) * s.heads + head) * L.bytes;
    uint8_t *dst = ring + c % stages * stage_bytes;
    uint64_t *bar = &full[c % stages];
    mbar_arrive_expect_tx(bar, stage_bytes);
    bulk_copy_g2s(dst, src, L.v, bar);
    bulk_copy_g2s(dst + L.v, src + L.v + slice * ItemLayout::slice_bytes(), ItemLayout::slice_bytes(), bar);
  };
  if (tid == 0)
    for (uint32_t c = 0; c < min(stages, por.chunks); ++c) issue(c);

  const uint32_t mt = warp & 3, half = warp >> 2;             // output: 16 rows, 16 columns per warp
  const uint32_t r8 = lane & 7, m1 = lane >> 3 & 1, m2 = lane >> 4;  // ldmatrix: row inside a matrix, matrix index bits
  bool ok = true;
  for (uint32_t c = 0; c < por.chunks; ++c) {
    const GlaChunk ch = chunks[por.chunk + c];
    if (!__all_sync(0xffffffffu, mbar_wait(&full[c % stages], c / stages & 1))) ok = false;
    const uint32_t q = smem_u32(ring + c % stages * stage_bytes), k = q + L.k, A = q + L.a, v = q + L.v;
    const uint32_t hi = smem_u32(parts + (c % copies) * 2 * part), lo = hi + part * 2;
    float o[2][4] = {};
    for (uint32_t ks = 0; ks <= mt; ++ks) {  // the blocks above the diagonal are zero
      uint32_t a[4], b[4];
      ldmatrix_x4(a, A + (mt * 16 + r8 + m1 * 8) * (kAStride * 2) + (ks * 16 + m2 * 8) * 2);
      ldmatrix_x4_trans(b, v + (ks * 16 + r8 + m1 * 8) * (kVStride * 2) + (half * 16 + m2 * 8) * 2);
      mma_bf16_16816(o[0], a, b[0], b[1]);
      mma_bf16_16816(o[1], a, b[2], b[3]);
    }
    for (uint32_t d0 = 0; d0 < L.dims; d0 += 16) {
      uint32_t a[4], b[4];
      const uint32_t at = (d0 + r8 + m1 * 8) * (kVStride * 2) + (half * 16 + m2 * 8) * 2;
      ldmatrix_x4(a, q + (mt * 16 + r8 + m1 * 8) * (L.row * 2) + (d0 + m2 * 8) * 2);
      ldmatrix_x4_trans(b, lo + at);
      mma_bf16_16816(o[0], a, b[0], b[1]);
      mma_bf16_16816(o[1], a, b[2], b[3]);
      ldmatrix_x4_trans(b, hi + at);
      mma_bf16_16816(o[0], a, b[0], b[1]);
      mma_bf16_16816(o[1], a, b[2], b[3]);
    }
    const float *decay = reinterpret_cast<const float *>(ring + c % stages * stage_bytes + L.decay);
#pragma unroll
    for (int dt = 0; dt < DT; ++dt) {
      const uint32_t d0 = (warp + kWarps * dt) * 16;
      if (d0 >= L.dims) continue;
      const float e0 = decay[d0 + g], e1 = decay[d0 + g + 8];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) S[dt][nt][0] *= e0, S[dt][nt][1] *= e0, S[dt][nt][2] *= e1, S[dt][nt][3] *= e1;
#pragma unroll
      for (uint32_t ks = 0; ks < kC / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4_trans(a, k + (ks * 16 + r8 + m2 * 8) * (L.row * 2) + (d0 + m1 * 8) * 2);
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
          uint32_t b[4];
          ldmatrix_x4_trans(b, v + (ks * 16 + r8 + m1 * 8) * (kVStride * 2) + (n2 * 16 + m2 * 8) * 2);
          mma_bf16_16816(S[dt][2 * n2], a, b[0], b[1]);
          mma_bf16_16816(S[dt][2 * n2 + 1], a, b[2], b[3]);
        }
      }
    }
    if (copies == 1) __syncthreads();  // everybody has read the one copy of the state
    publish((c + 1) % copies);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t t = mt * 16 + g + (e & 2 ? 8 : 0), col = v0 + half * 16 + nt * 8 + t2 + (e & 1);
        if (t < ch.count && col < s.value_dim) o_out[(size_t)(ch.row + t) * s.v_cols() + head * s.value_dim + col] = o[nt][e];
      }
    __syncthreads();  // the stage is free, the new state is there
    if (tid == 0 && c + stages < por.chunks) issue(c + stages);
  }
  each([&](float &x, uint32_t d, uint32_t v) {
    if (d < s.dim && v < s.value_dim) state[sb.write[por.seq] * s.state_floats() + base + (size_t)d * s.value_dim + v] = x;
  });
  if (!ok && lane == 0) atomicOr(&g_gla_error, 1u);
}

// Four heads of a chunk per CTA, a warp per row; values of at most 128 (VEC 4): the row's four heads are fetched at once.
template <int VEC, int SLABS>
__global__ void __launch_bounds__(kThreads)
gla_finish_kernel(const float *__restrict__ o, const float *__restrict__ partial, uint32_t splits, size_t split_stride, GlaShape s,
                  const float *__restrict__ norm, const GlaChunk *__restrict__ chunks, bf16 *__restrict__ out, uint32_t ldo) {
  pdl_trigger();
  const GlaChunk ch = chunks[blockIdx.x];
  const uint32_t lane = threadIdx.x & 31, h0 = blockIdx.y * 4, heads = min(4u, s.heads - h0), V = s.value_dim, v4 = lane * 4;
  const uint32_t g_at = 2 * s.q_cols() + s.v_cols();
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), w = VEC == 4 && v4 < V ? *reinterpret_cast<const float4 *>(norm + v4) : zero;
  pdl_wait();
  for (uint32_t n = threadIdx.x >> 5; n < ch.count; n += kWarps) {
    const uint32_t row = ch.row + n;
    const float *src = o + (size_t)row * s.v_cols() + h0 * V, *gate = partial + (size_t)row * s.ld + g_at + h0 * V;
    bf16 *dst = out + (size_t)row * ldo + h0 * V;
    if constexpr (VEC == 4) {
      float4 x[4], g[4];
#pragma unroll
      for (uint32_t h = 0; h < 4; ++h) {
        x[h] = g[h] = zero;
        if (h >= heads || v4 >= V) continue;
        x[h] = *reinterpret_cast<const float4 *>(src + h * V + v4);
        g[h] = sum_slabs4_most<SLABS>(gate + h * V + v4, splits, split_stride);
      }
#pragma unroll
      for (uint32_t h = 0; h < 4; ++h) {
        const float ss = warp_sum(x[h].x * x[h].x + x[h].y * x[h].y + x[h].z * x[h].z + x[h].w * x[h].w);
        const float scale = 1.0f / sqrtf(ss / (float)V + s.eps);
        if (h >= heads || v4 >= V) continue;
        *reinterpret_cast<uint2 *>(dst + h * V + v4) =
            make_uint2(pack_bf16x2(x[h].x * scale * w.x * silu_for<bf16>(g[h].x), x[h].y * scale * w.y * silu_for<bf16>(g[h].y)),
                       pack_bf16x2(x[h].z * scale * w.z * silu_for<bf16>(g[h].z), x[h].w * scale * w.w * silu_for<bf16>(g[h].w)));
      }
    } else {
      for (uint32_t h = 0; h < heads; ++h) {
        float ss = 0.f;
        for (uint32_t v = h * V + lane; v < (h + 1) * V; v += 32) ss += src[v] * src[v];
        const float scale = 1.0f / sqrtf(warp_sum(ss) / (float)V + s.eps);
        for (uint32_t v = lane; v < V; v += 32)
          dst[h * V + v] = __float2bfloat16_rn(src[h * V + v] * scale * norm[v] * silu_for<bf16>(fold_slabs(gate + h * V + v, splits, split_stride)));
      }
    }
  }
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

}  // namespace

bool gla_chunks_supported(GlaShape s) {
  return s.dim > 0 && s.dim <= 256 && s.value_dim > 0 && prepare_smem(s) <= kPrepareSmem && ScanPlan(s).smem > 0;
}

size_t gla_scratch_bytes(GlaShape s, uint32_t chunks, uint32_t rows) {
  return (size_t)chunks * s.heads * ItemLayout(s).bytes + (size_t)rows * s.v_cols() * sizeof(float);
}

int launch_gla_chunks(const float *partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<bf16> w, float *state, StateBatch sb,
                      GlaPortions p, void *scratch, bf16 *out, uint32_t ldo, cudaStream_t stream) {
  if (p.num_chunks == 0) return ORION_OK;
  if (!gla_chunks_supported(s)) return set_error(ORION_ERR_INTERNAL, "the chunked form of gated linear attention does not cover this shape");
  if (p.num_chunks > 65535 || p.num_portions > 65535) return set_error(ORION_ERR_INVALID_REQUEST, "too many prompt portions in one batch");
  const ItemLayout L(s);
  const ScanPlan plan(s);
  auto *items = static_cast<uint8_t *>(scratch);
  auto *o = reinterpret_cast<float *>(items + (size_t)p.num_chunks * s.heads * L.bytes);
  const bool vec = s.dim % 4 == 0 && s.value_dim % 4 == 0 && s.ld % 4 == 0 && split_stride % 4 == 0;
  const int slabs = splits <= 1 ? 1 : (splits <= 4 ? 4 : 0);
  auto pick = [&](auto any, auto one, auto four) { return slabs == 1 ? one : (slabs == 4 ? four : any); };
  static bool attr_set[6][kMaxDeviceOrdinals] = {};
  auto prepare = vec ? pick(gla_prepare_kernel<true, 0>, gla_prepare_kernel<true, 1>, gla_prepare_kernel<true, 4>) : gla_prepare_kernel<false, 0>;
  ORION_CUDA_CHECK("gla_prepare attr", ensure_dynamic_smem(prepare, kPrepareSmem, attr_set[vec ? (slabs + 1) / 2 : 3]));
  ORION_CUDA_CHECK("gla_prepare", launch_pdl(prepare, dim3(s.heads, p.num_chunks), dim3(kThreads), prepare_smem(s), stream, partial, splits, split_stride,
                                             s, w, p.chunks, items));
  ORION_TRY(after_launch("gla_prepare"));
  const bool wide = L.dims > kWarps * 16;
  auto scan = wide ? gla_scan_kernel<2> : gla_scan_kernel<1>;
  ORION_CUDA_CHECK("gla_scan attr", ensure_dynamic_smem(scan, 227 * 1024, attr_set[4 + wide]));
  ORION_CUDA_CHECK("gla_scan", launch_pdl(scan, dim3(s.heads * L.slices, p.num_portions), dim3(kThreads), (size_t)plan.smem, stream,
                                          (const uint8_t *)items, s, state, sb, p.chunks, p.portions, o, plan.stages, plan.copies));
  ORION_TRY(after_launch("gla_scan"));
  auto finish = vec && ldo % 4 == 0 && s.value_dim <= 128 ? pick(gla_finish_kernel<4, 0>, gla_finish_kernel<4, 1>, gla_finish_kernel<4, 4>)
                                                          : gla_finish_kernel<1, 0>;
  ORION_CUDA_CHECK("gla_finish", launch_pdl(finish, dim3(p.num_chunks, (s.heads + 3) / 4), dim3(kThreads), 0,
                                            stream, (const float *)o, partial, splits, split_stride, s, w.norm, p.chunks, out, ldo));
  return after_launch("gla_finish");
}

int gla_poll_error(uint32_t *code) {
  uint32_t v = 0;
  ORION_CUDA_CHECK("gla error word", cudaMemcpyFromSymbol(&v, g_gla_error, sizeof v));
  if (v) {
    uint32_t zero = 0;
    ORION_CUDA_CHECK("gla error word", cudaMemcpyToSymbol(g_gla_error, &zero, sizeof zero));
  }
  *code = v;
  return ORION_OK;
}

}  // namespace orion
