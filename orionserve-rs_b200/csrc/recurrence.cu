// Element-wise gated recurrences over the rows of each sequence, S_t = a_t S_(t-1) + b_t, with gates that read
// the current row only. All of it is f32: the gates' arguments are the projections' f32 partial sums, the
// state lives in f32 and is carried from step to step.
//   min_gru_step_kernel   one row per sequence (decode): four channels per thread
//   min_gru_scan_kernel   any batch: CTA = (32 channels, sequence); lanes are channels, each warp takes
//                         kRows consecutive rows of a tile, composes their maps S -> A S + B, the warps
//                         exchange (A, B) through shared memory, and each warp then runs its own rows from
//                         the state it starts at. The next tile's partial sums are in flight meanwhile. When
//                         there are too few (channels, sequences) to fill the machine, the CTAs of a cluster
//                         take consecutive tiles of one sequence and exchange their tiles' maps through
//                         distributed shared memory.
#include "kernels.h"

#include <algorithm>

namespace orion {
namespace {

// The map of one row and channel: S -> a S + b.
template <typename T>
__device__ __forceinline__ void min_gru_map(float z_pre, float x_pre, float &a, float &b) {
  const float z = sigmoid_for<T>(z_pre), below = sigmoid_for<T>(x_pre), cand = x_pre >= 0.f ? x_pre + 0.5f : below;
  a = 1.f - z;
  b = z * cand;
}

template <typename T>
__global__ void __launch_bounds__(128)
min_gru_step_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const float *__restrict__ bias,
                    float *__restrict__ state, StateBatch sb, T *__restrict__ out, uint32_t ldo, uint32_t width) {
  pdl_trigger();
  const uint32_t row = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f), bz = s, bx = s;
  const uint32_t rd = sb.read[row];
  if (c < width) {  // none of this is written by the preceding kernels of the step
    bz = *reinterpret_cast<const float4 *>(bias + c);
    bx = *reinterpret_cast<const float4 *>(bias + width + c);
    if (rd != kNoState) s = *reinterpret_cast<const float4 *>(state + (size_t)rd * width + c);
  }
  pdl_wait();
  if (c >= width) return;
  const float *p = partial + (size_t)row * 3 * width + c;
  const float4 z = sum_slabs4(p, splits, split_stride), x = sum_slabs4(p + width, splits, split_stride),
               g = sum_slabs4(p + 2 * (size_t)width, splits, split_stride);
  const float zz[4] = {z.x + bz.x, z.y + bz.y, z.z + bz.z, z.w + bz.w}, xx[4] = {x.x + bx.x, x.y + bx.y, x.z + bx.z, x.w + bx.w};
  const float gg[4] = {g.x, g.y, g.z, g.w};
  float ss[4] = {s.x, s.y, s.z, s.w};
  T *o = out + (size_t)row * ldo + c;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float a, b;
    min_gru_map<T>(zz[i], xx[i], a, b);
    ss[i] = a * ss[i] + b;
    o[i] = from_f32<T>(ss[i] * gg[i] * sigmoid_for<T>(gg[i]));
  }
  *reinterpret_cast<float4 *>(state + (size_t)sb.write[row] * width + c) = make_float4(ss[0], ss[1], ss[2], ss[3]);
}

constexpr uint32_t kRows = 4, kMaxWarps = 16, kMaxCluster = 8;  // rows per warp and tile, warps per CTA, CTAs per cluster

__device__ __forceinline__ void store_cluster(float2 *local, uint32_t rank, float2 v) {  // into the same place of CTA `rank`
  asm volatile(
      "{\n\t.reg .b32 a;\n\t"
      "mapa.shared::cluster.u32 a, %0, %1;\n\t"
      "st.shared::cluster.v2.f32 [a], {%2, %3};\n\t}" ::"r"(smem_u32(local)),
      "r"(rank), "f"(v.x), "f"(v.y)
      : "memory");
}
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <typename T>
__global__ void __launch_bounds__(32 * kMaxWarps, 2)
min_gru_scan_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const float *__restrict__ bias,
                    float *__restrict__ state, StateBatch sb, T *__restrict__ out, uint32_t ldo, uint32_t width) {
  __shared__ float2 maps[2][kMaxWarps][32];      // [tile parity][warp][channel]
  __shared__ float2 tiles[2][kMaxCluster][32];   // the same for the tiles of the cluster's CTAs
  const uint32_t ctas = gridDim.z, rank = blockIdx.z;  // the cluster spans the grid's z
  pdl_trigger();
  pdl_wait();
  const uint32_t seq = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  const uint32_t c = blockIdx.x * 32 + lane, first = sb.first_row[seq], end = sb.first_row[seq + 1];
  const bool live = c < width;
  const uint32_t rd = sb.read[seq];
  const float bz = live ? bias[c] : 0.f, bx = live ? bias[width + c] : 0.f;
  float s = live && rd != kNoState ? state[(size_t)rd * width + c] : 0.f;
  const size_t ld = 3 * (size_t)width;
  float z[kRows], x[kRows], g[kRows];
  auto fetch = [&](uint32_t row0) {
#pragma unroll
    for (uint32_t i = 0; i < kRows; ++i) {
      z[i] = x[i] = g[i] = 0.f;
      if (!live || row0 + i >= end) continue;
      const float *p = partial + (size_t)(row0 + i) * ld + c;
      z[i] = p[0], x[i] = p[width], g[i] = p[2 * (size_t)width];
      for (uint32_t k = 1; k < splits; ++k) {
        p += split_stride;
        z[i] += p[0], x[i] += p[width], g[i] += p[2 * (size_t)width];
      }
    }
  };
  const uint32_t step = ctas * warps * kRows, mine0 = (rank * warps + warp) * kRows;
  fetch(first + mine0);
  if (ctas > 1) cluster_sync();  // every CTA of the cluster has started before anyone stores into it
  uint32_t parity = 0;
  for (uint32_t t0 = first; t0 < end; t0 += step, parity ^= 1) {
    const uint32_t row0 = t0 + mine0;
    float a[kRows], b[kRows], gate[kRows], A = 1.f, B = 0.f;
#pragma unroll
    for (uint32_t i = 0; i < kRows; ++i) {
      a[i] = 1.f, b[i] = 0.f;
      if (row0 + i < end) min_gru_map<T>(z[i] + bz, x[i] + bx, a[i], b[i]);
      gate[i] = g[i];
      A *= a[i];
      B = a[i] * B + b[i];
    }
    fetch(row0 + step);
    maps[parity][warp][lane] = make_float2(A, B);
    __syncthreads();
    float mine = s;  // the state this warp's rows start from; every warp ends up with the last state of all tiles in s
    if (ctas > 1) {
      if (warp < ctas) {  // warp k tells CTA k
        float2 whole = make_float2(1.f, 0.f);
        for (uint32_t k = 0; k < warps; ++k) {
          const float2 m = maps[parity][k][lane];
          whole = make_float2(m.x * whole.x, m.x * whole.y + m.y);
        }
        store_cluster(&tiles[parity][rank][lane], warp, whole);
      }
      cluster_sync();
      float before = s;
      for (uint32_t k = 0; k < ctas; ++k) {
        const float2 m = tiles[parity][k][lane];
        if (k == rank) before = s;
        s = m.x * s + m.y;
      }
      mine = before;
      for (uint32_t k = 0; k < warp; ++k) {
        const float2 m = maps[parity][k][lane];
        mine = m.x * mine + m.y;
      }
    } else {
#pragma unroll 4
      for (uint32_t k = 0; k < warps; ++k) {
        const float2 m = maps[parity][k][lane];
        if (k == warp) mine = s;
        s = m.x * s + m.y;
      }
    }
#pragma unroll
    for (uint32_t i = 0; i < kRows; ++i) {
      mine = a[i] * mine + b[i];
      if (live && row0 + i < end) out[(size_t)(row0 + i) * ldo + c] = from_f32<T>(mine * gate[i] * sigmoid_for<T>(gate[i]));
    }
  }
  if (live && warp == 0 && rank == 0) state[(size_t)sb.write[seq] * width + c] = s;
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

}  // namespace

template <typename T>
int launch_min_gru(const float *partial, uint32_t splits, size_t split_stride, const float *bias, float *state, StateBatch sb,
                   T *out, uint32_t ldo, uint32_t width, cudaStream_t stream) {
  if (sb.rows == 0 || width == 0) return ORION_OK;
  if (sb.single && width % 4 == 0) {
    ORION_CUDA_CHECK("min_gru", launch_pdl(min_gru_step_kernel<T>, dim3(sb.rows, (width / 4 + 127) / 128), dim3(128), 0, stream, partial,
                                           splits, split_stride, bias, state, sb, out, ldo, width));
    return after_launch("min_gru");
  }
  // warps per CTA: enough for the mean sequence in one tile; CTAs per cluster: as long as they find tiles and places
  const uint32_t mean = (sb.rows + sb.seqs - 1) / sb.seqs, groups = (width + 31) / 32 * sb.seqs;
  uint32_t ctas = 1;
  while (ctas < kMaxCluster && 2 * ctas * groups <= 2 * 148 && 2 * ctas * kMaxWarps * kRows <= mean) ctas *= 2;
  const uint32_t warps = ctas > 1 ? kMaxWarps : std::min(kMaxWarps, std::max(1u, (mean + kRows - 1) / kRows));
  const dim3 grid((width + 31) / 32, sb.seqs, ctas);
  if (ctas > 1)
    ORION_CUDA_CHECK("min_gru", launch_pdl_cluster(min_gru_scan_kernel<T>, grid, dim3(32 * warps), dim3(1, 1, ctas), 0, stream, partial,
                                                   splits, split_stride, bias, state, sb, out, ldo, width));
  else
    ORION_CUDA_CHECK("min_gru", launch_pdl(min_gru_scan_kernel<T>, grid, dim3(32 * warps), 0, stream, partial, splits, split_stride, bias,
                                           state, sb, out, ldo, width));
  return after_launch("min_gru");
}
template int launch_min_gru<float>(const float *, uint32_t, size_t, const float *, float *, StateBatch, float *, uint32_t, uint32_t,
                                   cudaStream_t);
template int launch_min_gru<bf16>(const float *, uint32_t, size_t, const float *, float *, StateBatch, bf16 *, uint32_t, uint32_t,
                                  cudaStream_t);

}  // namespace orion
