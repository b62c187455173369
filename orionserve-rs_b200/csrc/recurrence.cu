// Element-wise gated recurrences over the rows of each sequence, S_t = a_t S_(t-1) + b_t, with gates that read
// the current row only. All of it is f32: the gates' arguments are the projections' f32 partial sums, the
// state lives in f32 and is carried from step to step.
//   min_gru_step_kernel   one row per sequence (decode): four channels per thread
//   min_gru_scan_kernel   any batch: CTA = (32 channels, sequence); lanes are channels, each warp takes
//                         kRows consecutive rows of a tile, composes their maps S -> A S + B, the warps
//                         exchange (A, B) through shared memory, and each warp then runs its own rows from
//                         the state it starts at. The next tile's partial sums are in flight meanwhile.
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

constexpr uint32_t kRows = 8;  // rows per warp and tile

template <typename T>
__global__ void __launch_bounds__(1024)
min_gru_scan_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const float *__restrict__ bias,
                    float *__restrict__ state, StateBatch sb, T *__restrict__ out, uint32_t ldo, uint32_t width) {
  __shared__ float2 maps[2][32][32];  // [tile parity][warp][channel]
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
  fetch(first + warp * kRows);
  uint32_t parity = 0;
  for (uint32_t t0 = first; t0 < end; t0 += warps * kRows, parity ^= 1) {
    const uint32_t row0 = t0 + warp * kRows;
    float a[kRows], b[kRows], gate[kRows], A = 1.f, B = 0.f;
#pragma unroll
    for (uint32_t i = 0; i < kRows; ++i) {
      a[i] = 1.f, b[i] = 0.f;
      if (row0 + i < end) min_gru_map<T>(z[i] + bz, x[i] + bx, a[i], b[i]);
      gate[i] = g[i];
      A *= a[i];
      B = a[i] * B + b[i];
    }
    fetch(row0 + warps * kRows);
    maps[parity][warp][lane] = make_float2(A, B);
    __syncthreads();
    float mine = s;  // the state this warp's rows start from; every warp ends up with the tile's last state in s
    for (uint32_t k = 0; k < warps; ++k) {
      const float2 m = maps[parity][k][lane];
      if (k == warp) mine = s;
      s = m.x * s + m.y;
    }
#pragma unroll
    for (uint32_t i = 0; i < kRows; ++i) {
      mine = a[i] * mine + b[i];
      if (live && row0 + i < end) out[(size_t)(row0 + i) * ldo + c] = from_f32<T>(mine * gate[i] * sigmoid_for<T>(gate[i]));
    }
  }
  if (live && warp == 0) state[(size_t)sb.write[seq] * width + c] = s;
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
  // warps per CTA: enough for the mean sequence in one tile, at most 32
  const uint32_t mean = (sb.rows + sb.seqs - 1) / sb.seqs;
  const uint32_t warps = std::min(32u, std::max(1u, (mean + kRows - 1) / kRows));
  ORION_CUDA_CHECK("min_gru", launch_pdl(min_gru_scan_kernel<T>, dim3((width + 31) / 32, sb.seqs), dim3(32 * warps), 0, stream, partial,
                                         splits, split_stride, bias, state, sb, out, ldo, width));
  return after_launch("min_gru");
}
template int launch_min_gru<float>(const float *, uint32_t, size_t, const float *, float *, StateBatch, float *, uint32_t, uint32_t,
                                   cudaStream_t);
template int launch_min_gru<bf16>(const float *, uint32_t, size_t, const float *, float *, StateBatch, bf16 *, uint32_t, uint32_t,
                                  cudaStream_t);

}  // namespace orion
