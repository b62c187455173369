// Latent attention: queries and keys meet in a per-head space that is a linear image of one small latent per
// token, plus one rotated key part shared by all heads; only the latent and the shared part are cached. The
// product with a key is evaluated in the latent space: q . (W_uk c) = (W_uk^T q) . c, and the weighted sum of
// values is W_uv applied to the weighted sum of latents, so a decode step reads the cache once for all heads.
//   latent_prepare_kernel            folds the joint projection: queries rotated, latent normalised and cached
//   latent_attention_generic_kernel  any shape and batch, f32 arithmetic: the f32 build and unusual shapes
#include "kernels.h"

#include <algorithm>

namespace orion {
namespace {

__device__ __forceinline__ float sigmoid_f(float x) {
  const float e = expf(-fabsf(x));
  return (x >= 0.f ? 1.f : e) / (1.f + e);
}
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
  const float *p = partial + (size_t)row * ls.cols();
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

constexpr uint32_t kGenThreads = 128, kGenKeys = 256;

template <typename T>
__global__ void __launch_bounds__(kGenThreads)
latent_attention_generic_kernel(const T *__restrict__ q, const T *__restrict__ cache, const T *__restrict__ w_uk,
                                const T *__restrict__ w_uv, const float *__restrict__ gate, uint32_t splits, size_t split_stride,
                                LatentShape ls, AttnBatch batch, T *__restrict__ out, uint32_t ldo) {
  extern __shared__ float smem[];
  float *q_s = smem;                     // [kv_rank + rot_dim]: the query in the latent space, then its rotated part
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
  const float *g = gate + (size_t)row * ls.cols() + ls.q_cols() + ls.kv_cols() + (size_t)head * ls.value_dim;
  T *o = out + (size_t)row * ldo + (size_t)head * ls.value_dim;
  for (uint32_t v = warp; v < ls.value_dim; v += kGenThreads / 32) {
    const T *w = w_uv + ((size_t)head * ls.value_dim + v) * ls.kv_rank;
    float a = 0.f;
    for (uint32_t r = lane; r < ls.kv_rank; r += 32) a += to_f32<T>(w[r]) * acc[r];
    a = warp_sum(a);
    if (lane == 0) o[v] = from_f32<T>(a * inv * sigmoid_f(fold(g + v, splits, split_stride)));
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

#define ORION_INSTANTIATE(T)                                                                                                        \
  template int launch_latent_prepare<T>(const float *, uint32_t, size_t, const float *, const float *, const float *, const uint32_t *, \
                                        const uint32_t *, const uint32_t *, T *, T *, LatentShape, uint32_t, cudaStream_t);           \
  template int launch_latent_attention_generic<T>(const T *, const T *, const T *, const T *, const float *, uint32_t, size_t,        \
                                                  LatentShape, AttnBatch, T *, uint32_t, cudaStream_t);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
