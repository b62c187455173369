// Short causal convolutions over time, one filter per channel, added to their input (h + conv(h)), with
// the last taps - 1 rows of h carried from step to step per sequence.
//   causal_conv_kernel          any batch; h comes from the norm kernel, neighbouring rows of a sequence from
//                               the batch itself, the rows before it from the sequence's state
//   residual_norm_conv_kernel   one row per sequence (decode): residual add or embedding lookup, norm and
//                               both convolutions in one pass over the row
// h is rounded to the storage type before the filters see it, in both kernels, so a row's result does not
// depend on whether its neighbours came from the batch or from the state.
#include "kernels.h"

#include <algorithm>

namespace orion {
namespace {

constexpr uint32_t kConvThreads = 128;

template <typename T>
__device__ __forceinline__ void load4(const T *p, float (&v)[4]);
template <>
__device__ __forceinline__ void load4<float>(const float *p, float (&v)[4]) {
  const float4 x = *reinterpret_cast<const float4 *>(p);
  v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
template <>
__device__ __forceinline__ void load4<bf16>(const bf16 *p, float (&v)[4]) {
  const uint2 x = *reinterpret_cast<const uint2 *>(p);
  v[0] = __uint_as_float(x.x << 16), v[1] = __uint_as_float(x.x & 0xFFFF0000u);
  v[2] = __uint_as_float(x.y << 16), v[3] = __uint_as_float(x.y & 0xFFFF0000u);
}
template <typename T>
__device__ __forceinline__ void store4(T *p, const float (&v)[4]);
template <>
__device__ __forceinline__ void store4<float>(float *p, const float (&v)[4]) {
  *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void store4<bf16>(bf16 *p, const float (&v)[4]) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
  uint2 x;
  x.x = *reinterpret_cast<const uint32_t *>(&lo);
  x.y = *reinterpret_cast<const uint32_t *>(&hi);
  *reinterpret_cast<uint2 *>(p) = x;
}
template <typename T, int N>
__device__ __forceinline__ void load_n(const T *p, float (&v)[N]) {
  if constexpr (N == 4) load4<T>(p, v);
  else v[0] = to_f32<T>(p[0]);
}
template <typename T, int N>
__device__ __forceinline__ void store_n(T *p, const float (&v)[N]) {
  if constexpr (N == 4) store4<T>(p, v);
  else p[0] = from_f32<T>(v[0]);
}

// VEC channels per thread (4, or 1 for widths that are no multiple of 4); blockIdx.x = batch row.
template <typename T, int VEC>
__global__ void __launch_bounds__(kConvThreads)
causal_conv_kernel(const T *__restrict__ h, const T *__restrict__ w1, const T *__restrict__ w2, uint32_t taps, T *__restrict__ state,
                   StateBatch sb, T *__restrict__ out1, T *__restrict__ out2, uint32_t cols) {
  pdl_trigger();
  pdl_wait();
  const uint32_t row = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  if (c >= cols) return;
  const uint32_t seq = sb.seq_of_row[row], first = sb.first_row[seq], last = sb.first_row[seq + 1] - 1;
  const uint32_t rd = sb.read[seq], keep = taps - 1, at = row - first;
  const T *old = state + (size_t)rd * keep * cols;  // looked at only if rd names a copy
  T *fresh = state + (size_t)sb.write[seq] * keep * cols;
  float x[VEC], a1[VEC], a2[VEC];
  load_n<T, VEC>(h + (size_t)row * cols + c, x);
#pragma unroll
  for (int i = 0; i < VEC; ++i) a1[i] = a2[i] = 0.f;
  for (uint32_t j = 0; j < taps; ++j) {
    const uint32_t lag = keep - j;
    float v[VEC];
    if (lag <= at) load_n<T, VEC>(h + (size_t)(row - lag) * cols + c, v);
    else if (rd != kNoState) load_n<T, VEC>(old + (size_t)(keep - (lag - at)) * cols + c, v);
    else continue;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      a1[i] += to_f32<T>(w1[(size_t)j * cols + c + i]) * v[i];
      if (w2) a2[i] += to_f32<T>(w2[(size_t)j * cols + c + i]) * v[i];
    }
  }
#pragma unroll
  for (int i = 0; i < VEC; ++i) a1[i] += x[i], a2[i] += x[i];
  store_n<T, VEC>(out1 + (size_t)row * cols + c, a1);
  if (w2) store_n<T, VEC>(out2 + (size_t)row * cols + c, a2);
  // the last taps - 1 rows are the next step's state; a sequence with fewer rows shifts the old ones down
  const uint32_t left = last - row, n = last - first + 1;
  if (left < keep) store_n<T, VEC>(fresh + (size_t)(keep - 1 - left) * cols + c, x);
  if (at == 0)
    for (uint32_t k = 0; k + n < keep; ++k) {
      float v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) v[i] = 0.f;
      if (rd != kNoState) load_n<T, VEC>(old + (size_t)(k + n) * cols + c, v);
      store_n<T, VEC>(fresh + (size_t)k * cols + c, v);
    }
}

// The same for TAPS filters' taps known at compile time: four channels and eight rows per thread, the filters and
// the last TAPS - 1 rows in registers, the tile's rows in flight together. blockIdx.x = tile of eight rows.
constexpr uint32_t kConvRows = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads)
causal_conv_tile_kernel(const T *__restrict__ h, const T *__restrict__ w1, const T *__restrict__ w2, T *__restrict__ state, StateBatch sb,
                        T *__restrict__ out1, T *__restrict__ out2, uint32_t cols) {
  constexpr uint32_t kKeep = TAPS - 1;
  pdl_trigger();
  const uint32_t row0 = blockIdx.x * kConvRows, c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
  if (c >= cols) {
    pdl_wait();
    return;
  }
  float f1[TAPS][4], f2[TAPS][4];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {  // filters are immutable
    load4<T>(w1 + (size_t)j * cols + c, f1[j]);
    if (w2) load4<T>(w2 + (size_t)j * cols + c, f2[j]);
  }
  pdl_wait();
  float x[kConvRows][4], past[TAPS][4];  // past[k]: k + 1 rows back; the last entry pads the shift
#pragma unroll
  for (uint32_t i = 0; i < kConvRows; ++i)
    if (row0 + i < sb.rows) load4<T>(h + (size_t)(row0 + i) * cols + c, x[i]);
  uint32_t seq = kNoState, first = 0, last = 0, rd = kNoState;
  const T *old = state;
  T *fresh = state;
#pragma unroll
  for (uint32_t i = 0; i < kConvRows; ++i) {
    const uint32_t row = row0 + i;
    if (row >= sb.rows) break;
    if (seq == kNoState || row > last) {  // another sequence: its rows before this one come from the batch or the state
      seq = sb.seq_of_row[row], first = sb.first_row[seq], last = sb.first_row[seq + 1] - 1, rd = sb.read[seq];
      old = state + (size_t)(rd == kNoState ? 0 : rd) * kKeep * cols + c;
      fresh = state + (size_t)sb.write[seq] * kKeep * cols + c;
#pragma unroll
      for (uint32_t k = 0; k < kKeep; ++k) {
        const uint32_t lag = k + 1, at = row - first;
        past[k][0] = past[k][1] = past[k][2] = past[k][3] = 0.f;
        if (lag <= at) load4<T>(h + (size_t)(row - lag) * cols + c, past[k]);
        else if (rd != kNoState) load4<T>(old + (size_t)(kKeep - (lag - at)) * cols, past[k]);
      }
    }
    float a1[4], a2[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      a1[e] = f1[kKeep][e] * x[i][e] + x[i][e];
      a2[e] = w2 ? f2[kKeep][e] * x[i][e] + x[i][e] : 0.f;
#pragma unroll
      for (uint32_t k = 0; k < kKeep; ++k) {
        a1[e] += f1[kKeep - 1 - k][e] * past[k][e];
        if (w2) a2[e] += f2[kKeep - 1 - k][e] * past[k][e];
      }
    }
    store4<T>(out1 + (size_t)row * cols + c, a1);
    if (w2) store4<T>(out2 + (size_t)row * cols + c, a2);
    const uint32_t left = last - row, n = last - first + 1;
    if (left < kKeep) store4<T>(fresh + (size_t)(kKeep - 1 - left) * cols, x[i]);
    if (row == first)  // a sequence with fewer rows than the state holds shifts the old ones down
      for (uint32_t k = 0; k + n < kKeep; ++k) {
        float v[4] = {0.f, 0.f, 0.f, 0.f};
        if (rd != kNoState) load4<T>(old + (size_t)(k + n) * cols, v);
        store4<T>(fresh + (size_t)k * cols, v);
      }
#pragma unroll
    for (int k = (int)kKeep - 1; k > 0; --k)
#pragma unroll
      for (int e = 0; e < 4; ++e) past[k][e] = past[k - 1][e];
#pragma unroll
    for (int e = 0; e < 4; ++e) past[0][e] = x[i][e];
  }
}

template <typename T>
struct SumOf { using type = float; };
template <>
struct SumOf<float> { using type = double; };

// Four channels as they are stored.
template <typename T>
struct Raw4 { using type = uint2; };
template <>
struct Raw4<float> { using type = float4; };
template <typename T>
__device__ __forceinline__ void unpack4(const typename Raw4<T>::type &x, float (&v)[4]) { load4<T>(reinterpret_cast<const T *>(&x), v); }

// One CTA per row, CHUNKS groups of four channels per thread. With TAPS > 0 the filters and the state, which no
// kernel of this step has written, are fetched before the wait for the preceding kernel; TAPS = 0 takes any number.
template <typename T, int CHUNKS, int TAPS>
__global__ void __launch_bounds__(1024)
residual_norm_conv_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, const T *__restrict__ embed,
                          const uint32_t *__restrict__ tokens, float *__restrict__ hidden, const float *__restrict__ norm_w, float eps,
                          const T *__restrict__ w1, const T *__restrict__ w2, uint32_t taps, T *__restrict__ state, StateBatch sb,
                          T *__restrict__ out1, T *__restrict__ out2, uint32_t cols) {
  using Acc = typename SumOf<T>::type;
  using Raw = typename Raw4<T>::type;
  constexpr int kTaps = TAPS > 0 ? TAPS : 1;
  __shared__ Acc red[32];
  pdl_trigger();
  const uint32_t row = blockIdx.x, nvec = cols / 4, keep = TAPS > 0 ? TAPS - 1 : taps - 1, rd = sb.read[row];
  const T *old = state + (size_t)(rd == kNoState ? 0 : rd) * keep * cols;
  T *fresh = state + (size_t)sb.write[row] * keep * cols;
  Raw past[CHUNKS][kTaps], f1[CHUNKS][kTaps], f2[CHUNKS][kTaps];
  if (TAPS > 0) {
#pragma unroll
    for (int k = 0; k < CHUNKS; ++k) {
      const uint32_t idx = threadIdx.x + k * blockDim.x;
      if (idx >= nvec) continue;
#pragma unroll
      for (int j = 0; j < kTaps; ++j) {
        f1[k][j] = *reinterpret_cast<const Raw *>(w1 + (size_t)j * cols + 4 * idx);
        if (w2) f2[k][j] = *reinterpret_cast<const Raw *>(w2 + (size_t)j * cols + 4 * idx);
        if (j + 1 < kTaps && rd != kNoState) past[k][j] = *reinterpret_cast<const Raw *>(old + (size_t)j * cols + 4 * idx);
      }
    }
  }
  pdl_wait();
  float v[CHUNKS][4];
  Acc ss = Acc(0);
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const uint32_t idx = threadIdx.x + k * blockDim.x;
    v[k][0] = v[k][1] = v[k][2] = v[k][3] = 0.f;
    if (idx >= nvec) continue;
    float *hp = hidden + (size_t)row * cols + 4 * idx;
    if (embed) {
      load4<T>(embed + (size_t)tokens[row] * cols + 4 * idx, v[k]);
    } else {
      const float4 r = *reinterpret_cast<const float4 *>(hp);
      const float4 add = sum_slabs4(partial + (size_t)row * cols + 4 * idx, splits, split_stride);
      v[k][0] = r.x + add.x, v[k][1] = r.y + add.y, v[k][2] = r.z + add.z, v[k][3] = r.w + add.w;
    }
    *reinterpret_cast<float4 *>(hp) = make_float4(v[k][0], v[k][1], v[k][2], v[k][3]);
#pragma unroll
    for (int i = 0; i < 4; ++i) ss += (Acc)v[k][i] * (Acc)v[k][i];
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  Acc total = Acc(0);
  for (uint32_t i = 0; i < (blockDim.x + 31) / 32; ++i) total += red[i];
  float scale;
  if constexpr (sizeof(T) == 4) scale = (float)(1.0 / sqrt(total / (double)cols + (double)eps));
  else scale = rsqrtf(total / (float)cols + eps);
#pragma unroll
  for (int k = 0; k < CHUNKS; ++k) {
    const uint32_t idx = threadIdx.x + k * blockDim.x;
    if (idx >= nvec) continue;
    const uint32_t c = 4 * idx;
    const float4 g = *reinterpret_cast<const float4 *>(norm_w + c);
    float x[4] = {v[k][0] * scale * g.x, v[k][1] * scale * g.y, v[k][2] * scale * g.z, v[k][3] * scale * g.w};
    float a1[4], a2[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) a1[i] = a2[i] = x[i] = to_f32<T>(from_f32<T>(x[i]));
    // tap j meets the row keep - j back: the state's row j, or this row for the last tap
    auto tap = [&](uint32_t j, const Raw &r1, const Raw &r2, const float (&o)[4]) {
      float w[4];
      unpack4<T>(r1, w);
#pragma unroll
      for (int i = 0; i < 4; ++i) a1[i] += w[i] * o[i];
      if (w2) {
        unpack4<T>(r2, w);
#pragma unroll
        for (int i = 0; i < 4; ++i) a2[i] += w[i] * o[i];
      }
      if (j > 0) store4<T>(fresh + (size_t)(j - 1) * cols + c, o);
    };
    if (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < kTaps; ++j) {
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if (j + 1 < kTaps && rd != kNoState) unpack4<T>(past[k][j], o);
        tap(j, f1[k][j], f2[k][j], j + 1 < kTaps ? o : x);
      }
    } else {
      for (uint32_t j = 0; j <= keep; ++j) {
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if (j < keep && rd != kNoState) load4<T>(old + (size_t)j * cols + c, o);
        tap(j, *reinterpret_cast<const Raw *>(w1 + (size_t)j * cols + c), *reinterpret_cast<const Raw *>((w2 ? w2 : w1) + (size_t)j * cols + c),
            j < keep ? o : x);
      }
    }
    store4<T>(out1 + (size_t)row * cols + c, a1);
    if (w2) store4<T>(out2 + (size_t)row * cols + c, a2);
  }
}

template <typename T>
__global__ void transpose_kernel(const T *__restrict__ src, T *__restrict__ dst, uint32_t rows, uint32_t cols) {
  for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < rows * cols; i += gridDim.x * blockDim.x)
    dst[(size_t)(i % cols) * rows + i / cols] = src[i];
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

}  // namespace

template <typename T>
int launch_causal_conv(const T *h, const T *w1, const T *w2, uint32_t taps, T *state, StateBatch sb, T *out1, T *out2,
                       uint32_t cols, cudaStream_t stream) {
  if (sb.rows == 0) return ORION_OK;
  if (cols % 4 == 0 && taps >= 2 && taps <= 4) {
    const dim3 grid((sb.rows + kConvRows - 1) / kConvRows, (cols / 4 + kConvThreads - 1) / kConvThreads);
    auto kernel = taps == 2 ? causal_conv_tile_kernel<T, 2> : (taps == 3 ? causal_conv_tile_kernel<T, 3> : causal_conv_tile_kernel<T, 4>);
    ORION_CUDA_CHECK("causal_conv", launch_pdl(kernel, grid, dim3(kConvThreads), 0, stream, h, w1, w2, state, sb, out1, out2, cols));
    return after_launch("causal_conv");
  }
  const bool vec = cols % 4 == 0;
  const uint32_t per = kConvThreads * (vec ? 4 : 1);
  const dim3 grid(sb.rows, (cols + per - 1) / per);
  ORION_CUDA_CHECK("causal_conv", launch_pdl(vec ? causal_conv_kernel<T, 4> : causal_conv_kernel<T, 1>, grid, dim3(kConvThreads), 0,
                                             stream, h, w1, w2, taps, state, sb, out1, out2, cols));
  return after_launch("causal_conv");
}

bool residual_norm_conv_supported(uint32_t cols, uint32_t taps) { return taps >= 1 && cols % 4 == 0 && cols / 4 <= 4096; }

template <typename T>
int launch_residual_norm_conv(const float *partial, uint32_t splits, size_t split_stride, const T *embed, const uint32_t *tokens,
                              float *hidden, const float *norm_w, float eps, const T *w1, const T *w2, uint32_t taps, T *state,
                              StateBatch sb, T *out1, T *out2, uint32_t cols, cudaStream_t stream) {
  if (sb.rows == 0) return ORION_OK;
  if (!sb.single || !residual_norm_conv_supported(cols, taps))
    return set_error(ORION_ERR_INTERNAL, "the fused norm and convolution kernel does not cover this batch");
  const uint32_t nvec = cols / 4, threads = nvec >= 1024 ? 1024 : (nvec + 31) / 32 * 32, chunks = (nvec + threads - 1) / threads;
  auto kernel = chunks == 1 ? (taps == 4 ? residual_norm_conv_kernel<T, 1, 4> : residual_norm_conv_kernel<T, 1, 0>)
                            : (chunks == 2 ? residual_norm_conv_kernel<T, 2, 0> : residual_norm_conv_kernel<T, 4, 0>);
  ORION_CUDA_CHECK("residual_norm_conv", launch_pdl(kernel, dim3(sb.rows), dim3(threads), 0, stream, partial, splits, split_stride,
                                                    embed, tokens, hidden, norm_w, eps, w1, w2, taps, state, sb, out1, out2, cols));
  return after_launch("residual_norm_conv");
}

template <typename T>
int launch_transpose(const T *src, T *dst, uint32_t rows, uint32_t cols, cudaStream_t stream) {
  if (rows == 0 || cols == 0) return ORION_OK;
  transpose_kernel<T><<<std::min((rows * cols + 255) / 256, 148u * 16u), 256, 0, stream>>>(src, dst, rows, cols);
  return after_launch("transpose");
}

#define ORION_INSTANTIATE(T)                                                                                                      \
  template int launch_causal_conv<T>(const T *, const T *, const T *, uint32_t, T *, StateBatch, T *, T *, uint32_t, cudaStream_t); \
  template int launch_transpose<T>(const T *, T *, uint32_t, uint32_t, cudaStream_t);                                               \
  template int launch_residual_norm_conv<T>(const float *, uint32_t, size_t, const T *, const uint32_t *, float *, const float *, float, \
                                            const T *, const T *, uint32_t, T *, StateBatch, T *, T *, uint32_t, cudaStream_t);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
