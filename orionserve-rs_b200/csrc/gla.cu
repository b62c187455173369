// Gated linear attention, S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head, token by token. All of it is f32: the
// operands are the projections' f32 partial sums, the decays are formed here, the state lives in f32.
//   gla_step_kernel     one CTA per (head, sequence): the head's state stays in registers, four value columns by ROWS key rows per
//                       thread, while the sequence's rows of the batch pass by; the norm over the head and the gate end each row
//   gla_generic_kernel  the same for sizes that the registers do not take: a thread per value column, the state in its slot
// gla_chunk.cu has the form for prompt portions.
#include "gla.cuh"

#include <algorithm>

namespace orion {
namespace {

constexpr uint32_t kThreads = 256;

// What one row needs, folded into shared memory by the whole CTA: q (scaled), k and alpha of the head, its v and gate input.
template <typename T>
struct RowInputs {
  float *q, *k, *alpha, *v, *g, *a;
  T *decay;  // the head's decay weights where they are few, else null
  __device__ RowInputs(float *smem, const GlaShape &s)
      : q(smem), k(q + s.dim), alpha(k + s.dim), v(alpha + s.dim), g(v + s.value_dim), a(g + s.value_dim),
        decay(held(s) ? reinterpret_cast<T *>(smem + (values(s) + 3) / 4 * 4) : nullptr) {}
  static __host__ __device__ size_t values(const GlaShape &s) { return 3 * (size_t)s.dim + 2 * (size_t)s.value_dim + s.rank; }
  static __host__ __device__ size_t held(const GlaShape &s) { return s.dim * s.rank <= 4096 ? s.dim * s.rank : 0; }
  static __host__ __device__ size_t floats(const GlaShape &s) { return (values(s) + 3) / 4 * 4 + (held(s) * sizeof(T) + 15) / 16 * 4; }

  // Weights: before the kernel waits for the projection.
  __device__ void fetch_weights(const GlaShape &s, const GlaWeights<T> &w, uint32_t head) const {
    if (decay)
      for (uint32_t i = threadIdx.x; i < s.dim * s.rank; i += blockDim.x) decay[i] = w.decay[(size_t)head * s.dim * s.rank + i];
  }

  __device__ void load(const float *p, uint32_t splits, size_t stride, const GlaShape &s, const GlaWeights<T> &w, uint32_t head) const {
    const uint32_t nq = s.q_cols(), nv = s.v_cols(), D = s.dim, V = s.value_dim, all = 2 * D + 2 * V + s.rank;
    const float qs = 1.0f / sqrtf((float)D);
    for (uint32_t i0 = threadIdx.x; i0 < all; i0 += 2 * blockDim.x) {  // two at a time: their loads overlap
      float x[2], *dst[2];
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        const uint32_t i = i0 + u * blockDim.x;
        uint32_t at = 0;
        dst[u] = nullptr;
        if (i < D) at = head * D + i, dst[u] = q + i;
        else if (i < 2 * D) at = nq + head * D + (i - D), dst[u] = k + (i - D);
        else if (i < 2 * D + V) at = 2 * nq + head * V + (i - 2 * D), dst[u] = v + (i - 2 * D);
        else if (i < 2 * D + 2 * V) at = 2 * nq + nv + head * V + (i - 2 * D - V), dst[u] = g + (i - 2 * D - V);
        else if (i < all) at = 2 * nq + 2 * nv + (i - 2 * D - 2 * V), dst[u] = a + (i - 2 * D - 2 * V);
        x[u] = dst[u] ? fold_slabs(p + at, splits, stride) * (i < D ? qs : 1.f) : 0.f;
      }
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (dst[u]) *dst[u] = x[u];
    }
    __syncthreads();
    // four lanes per channel, every fourth weight each
    const T *wd = decay ? decay : w.decay + (size_t)head * D * s.rank;
    for (uint32_t d0 = 0; d0 < D; d0 += blockDim.x / 4) {
      const uint32_t d = d0 + threadIdx.x / 4, part = threadIdx.x & 3;
      float z = 0.f;
      if (d < D)
        for (uint32_t r = part; r < s.rank; r += 4) z = fmaf(to_f32<T>(wd[d * s.rank + r]), a[r], z);
      z += __shfl_xor_sync(0xffffffffu, z, 1);
      z += __shfl_xor_sync(0xffffffffu, z, 2);
      if (d < D && part == 0) alpha[d] = expf(log_sigmoid_for<T>(z + w.bias[(size_t)head * D + d]) / s.tau);
    }
    __syncthreads();
  }
};

// The head's output: o over its root mean square, times the gain, times silu of the gate's input. o in shared memory.
template <typename T>
__device__ __forceinline__ void finish_head(const float *o, const float *g, const GlaShape &s, const float *norm, float *red, T *out) {
  float ss = 0.f;
  for (uint32_t v = threadIdx.x; v < s.value_dim; v += blockDim.x) ss += o[v] * o[v];
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = 0.f;
  for (uint32_t w = 0; w < blockDim.x / 32; ++w) total += red[w];
  const float scale = 1.0f / sqrtf(total / (float)s.value_dim + s.eps);
  for (uint32_t v = threadIdx.x; v < s.value_dim; v += blockDim.x) out[v] = from_f32<T>(o[v] * scale * norm[v] * silu_for<T>(g[v]));
}

template <typename T, int ROWS>
__global__ void __launch_bounds__(kThreads, ROWS <= 8 ? 4 : 2)
gla_step_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<T> w, float *__restrict__ state,
                StateBatch sb, uint32_t most_rows, T *__restrict__ out, uint32_t ldo) {
  extern __shared__ float smem[];
  __shared__ float red[kThreads / 32];
  const RowInputs<T> in(smem, s);
  float *sums = smem + RowInputs<T>::floats(s);  // [key groups][value_dim]
  pdl_trigger();
  const uint32_t head = blockIdx.x, seq = blockIdx.y, first = sb.first_row[seq], end = sb.first_row[seq + 1];
  if (end - first > most_rows) {
    pdl_wait();  // what follows this grid relies on it having waited
    return;
  }
  const uint32_t cols = s.value_dim / 4, groups = kThreads / cols, col = threadIdx.x % cols, group = threadIdx.x / cols;
  const size_t at = (size_t)head * s.dim * s.value_dim + 4 * col;
  const uint32_t rd = sb.read[seq];
  float4 S[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {  // written by an earlier step: need not wait for this one's kernels
    const uint32_t d = group + i * groups;
    S[i] = rd != kNoState && group < groups && d < s.dim
               ? *reinterpret_cast<const float4 *>(state + rd * s.state_floats() + at + (size_t)d * s.value_dim)
               : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  in.fetch_weights(s, w, head);
  pdl_wait();
  for (uint32_t row = first; row < end; ++row) {
    in.load(partial + (size_t)row * s.ld, splits, split_stride, s, w, head);
    const float4 v = *reinterpret_cast<const float4 *>(in.v + 4 * col);
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const uint32_t d = group + i * groups;
      if (group >= groups || d >= s.dim) continue;
      const float a = in.alpha[d], k = in.k[d], q = in.q[d];
      S[i] = make_float4(a * S[i].x + k * v.x, a * S[i].y + k * v.y, a * S[i].z + k * v.z, a * S[i].w + k * v.w);
      o = make_float4(o.x + q * S[i].x, o.y + q * S[i].y, o.z + q * S[i].z, o.w + q * S[i].w);
    }
    if (group < groups) *reinterpret_cast<float4 *>(sums + (size_t)group * s.value_dim + 4 * col) = o;
    __syncthreads();
    for (uint32_t c = threadIdx.x; c < s.value_dim; c += kThreads) {  // each column is read and written by one thread
      float t = sums[c];
      for (uint32_t k = 1; k < groups; ++k) t += sums[(size_t)k * s.value_dim + c];
      sums[c] = t;
    }
    finish_head<T>(sums, in.g, s, w.norm, red, out + (size_t)row * ldo + head * s.value_dim);
    __syncthreads();
  }
  float *dst = state + sb.write[seq] * s.state_floats() + at;
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const uint32_t d = group + i * groups;
    if (group < groups && d < s.dim) *reinterpret_cast<float4 *>(dst + (size_t)d * s.value_dim) = S[i];
  }
}

template <typename T>
__global__ void __launch_bounds__(kThreads)
gla_generic_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<T> w, float *__restrict__ state,
                   StateBatch sb, uint32_t most_rows, T *__restrict__ out, uint32_t ldo) {
  extern __shared__ float smem[];
  __shared__ float red[kThreads / 32];
  const RowInputs<T> in(smem, s);
  float *sums = smem + RowInputs<T>::floats(s);  // [value_dim]
  pdl_trigger();
  in.fetch_weights(s, w, blockIdx.x);
  pdl_wait();
  const uint32_t head = blockIdx.x, seq = blockIdx.y, first = sb.first_row[seq], end = sb.first_row[seq + 1], V = s.value_dim;
  if (end - first > most_rows) return;
  const uint32_t rd = sb.read[seq];
  const size_t at = (size_t)head * s.dim * V;
  float *mine = state + sb.write[seq] * s.state_floats() + at;
  const float *before = rd != kNoState ? state + rd * s.state_floats() + at : nullptr;
  for (uint32_t row = first; row < end; ++row, before = mine) {
    in.load(partial + (size_t)row * s.ld, splits, split_stride, s, w, head);
    for (uint32_t c = threadIdx.x; c < V; c += kThreads) {
      const float v = in.v[c];
      float o = 0.f;
#pragma unroll 8
      for (uint32_t d = 0; d < s.dim; ++d) {
        const float x = in.alpha[d] * (before ? before[(size_t)d * V + c] : 0.f) + in.k[d] * v;
        mine[(size_t)d * V + c] = x;
        o += in.q[d] * x;
      }
      sums[c] = o;
    }
    finish_head<T>(sums, in.g, s, w.norm, red, out + (size_t)row * ldo + head * V);
    __syncthreads();
  }
}

}  // namespace

template <typename T>
int launch_gla_steps(const float *partial, uint32_t splits, size_t split_stride, GlaShape s, GlaWeights<T> w, float *state, StateBatch sb,
                     uint32_t most_rows, T *out, uint32_t ldo, cudaStream_t stream) {
  if (sb.rows == 0) return ORION_OK;
  const uint32_t cols = s.value_dim / 4, groups = s.value_dim % 4 == 0 && cols <= kThreads ? kThreads / cols : 0;
  const uint32_t each = groups ? (s.dim + groups - 1) / groups : UINT32_MAX;  // key rows per thread
  auto kernel = each <= 4 ? gla_step_kernel<T, 4> : (each <= 8 ? gla_step_kernel<T, 8> : (each <= 16 ? gla_step_kernel<T, 16> : gla_generic_kernel<T>));
  // float4 accesses to v: it starts at a multiple of four
  const bool vec = each <= 16 && s.dim % 4 == 0;
  if (!vec) kernel = gla_generic_kernel<T>;
  const size_t smem = (RowInputs<T>::floats(s) + (size_t)(vec ? groups : 1) * s.value_dim) * sizeof(float);
  if (smem > 48 * 1024) return set_error(ORION_ERR_INTERNAL, "gated linear attention with heads of %u x %u values is not supported", s.dim, s.value_dim);
  ORION_CUDA_CHECK("gla", launch_pdl(kernel, dim3(s.heads, sb.seqs), dim3(kThreads), smem, stream, partial, splits, split_stride, s, w, state, sb,
                                     most_rows, out, ldo));
  count_launch();
  ORION_CUDA_CHECK("gla", cudaGetLastError());
  return ORION_OK;
}
template int launch_gla_steps<float>(const float *, uint32_t, size_t, GlaShape, GlaWeights<float>, float *, StateBatch, uint32_t, float *, uint32_t,
                                     cudaStream_t);
template int launch_gla_steps<bf16>(const float *, uint32_t, size_t, GlaShape, GlaWeights<bf16>, float *, StateBatch, uint32_t, bf16 *, uint32_t,
                                    cudaStream_t);

}  // namespace orion
