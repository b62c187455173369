// What attention with query / key norms, rotation of part of each head and output gates needs between its joint projection
// and the attention kernels: one pass over the projection's partial sums that normalises, rotates, and leaves queries, cached
// keys and values, and gates. One CTA per row where a norm spans all heads, one warp per row and head where it does not. Where the
// values are the keys before their norm, the cache gets them once, beside the factor of that norm.
#include "kernels.h"
#include "mma.cuh"

namespace orion {
namespace {

__device__ __forceinline__ float fold(const float *p, uint32_t splits, size_t stride) {
  float v = p[0];
  for (uint32_t s = 1; s < splits; ++s) v += p[s * stride];
  return v;
}

// Sums of two values over the CTA (at most 32 warps), the same in every thread.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2 *red) {
  a = warp_sum(a), b = warp_sum(b);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  for (uint32_t w = 0; w < blockDim.x / 32; ++w) t.x += red[w].x, t.y += red[w].y;
  return t;
}

// Any sizes, one column at a time; the partial sums are folded once for the norms and once for the values.
template <typename T>
__global__ void __launch_bounds__(256)
attention_prepare_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, AttnInputs in,
                         const uint32_t *__restrict__ positions, const uint32_t *__restrict__ slot_block,
                         const uint32_t *__restrict__ slot_slot, T *__restrict__ q_out, T *__restrict__ arena, KvLayout kv, uint32_t layer,
                         float *__restrict__ gate) {
  __shared__ float2 red[32];
  pdl_trigger();
  pdl_wait();
  const uint32_t row = blockIdx.x, tid = threadIdx.x, half = in.rope_dims / 2;
  const float *p = partial + (size_t)row * in.ld;
  const uint32_t nq = in.q_heads * in.dim, nk = in.kv_heads * in.dim, nv = in.keys_as_values ? 0 : in.kv_heads * in.value_dim;
  float sq = 0.f, sk = 0.f;
  auto projected = [&](uint32_t i) { return fold(p + i, splits, split_stride) + (in.bias ? in.bias[i] : 0.f); };
  for (uint32_t i = tid; i < nq + nk; i += blockDim.x) {
    const float v = projected(i);
    if (i < nq) sq += v * v;
    else sk += v * v;
  }
  const float2 ss = block_sum2(sq, sk, red);
  const float scale_q = 1.0f / sqrtf(ss.x / (float)nq + in.eps), scale_k = 1.0f / sqrtf(ss.y / (float)nk + in.eps);
  const float *cs = in.rope_cos + (size_t)positions[row] * half, *sn = in.rope_sin + (size_t)positions[row] * half;
  const uint32_t block = slot_block[row], slot = slot_slot[row];
  if (in.keys_as_values) {
    const float factor = in.q_factor ? in.q_factor[positions[row]] * scale_q : scale_q;
    for (uint32_t i = tid; i < nq + nk; i += blockDim.x) {
      const float v = projected(i);
      const uint32_t c = i < nq ? i : i - nq, head = c / in.dim, d = c % in.dim;
      if (i < nq) q_out[((size_t)row * in.q_heads + head) * kv.head_dim + d] = from_f32<T>(v * factor * in.q_norm[i]);
      else arena[kv.row(layer, block, head, 0, slot) + kv.col(slot, d)] = from_f32<T>(v);
    }
    for (uint32_t h = tid; h < in.kv_heads; h += blockDim.x) *reinterpret_cast<float *>(arena + kv.factor(layer, block, h, slot)) = scale_k;
    return;
  }
  for (uint32_t i = tid; i < nq + nk; i += blockDim.x) {
    const bool is_q = i < nq;
    const uint32_t c = is_q ? i : i - nq, head = c / in.dim, d = c % in.dim;
    const float *w = is_q ? in.q_norm : in.k_norm;
    const float scale = is_q ? scale_q : scale_k;
    auto value = [&](uint32_t at) { return w ? projected(at) * scale * w[is_q ? at : at - nq] : projected(at); };
    float v = value(i);
    if (d < 2 * half) {
      const float other = value((d & 1) ? i - 1 : i + 1), co = cs[d >> 1], si = sn[d >> 1];
      v = (d & 1) ? v * co + other * si : v * co - other * si;
    }
    if (is_q) q_out[((size_t)row * in.q_heads + head) * kv.head_dim + d] = from_f32<T>(v);
    else arena[kv.row(layer, block, head, 0, slot) + kv.col(slot, d)] = from_f32<T>(v);
  }
  for (uint32_t i = tid; i < nv; i += blockDim.x)
    arena[kv.row(layer, block, i / in.value_dim, 1, slot) + kv.col(slot, i % in.value_dim)] = from_f32<T>(fold(p + nq + nk + i, splits, split_stride));
  if (gate)
    for (uint32_t h = tid; h < in.q_heads; h += blockDim.x)
      gate[(size_t)row * in.q_heads + h] = sigmoid_f(fold(p + nq + nk + nv + h, splits, split_stride));
}

template <typename T>
__device__ __forceinline__ void store4(T *p, float4 v);
template <>
__device__ __forceinline__ void store4<float>(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
template <>
__device__ __forceinline__ void store4<bf16>(bf16 *p, float4 v) {
  *reinterpret_cast<uint2 *>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// The same, four columns per thread and GROUPS rounds kept in registers, so each partial sum is read once: every size and
// stride a multiple of four. SLABS: the projection has at most that many (prompts; 0 = any number); gains and angles are then
// read when they are needed, not while the projection is still running, which leaves registers for more rows per SM. KEYS: keys as
// values, with biases.
template <typename T, int GROUPS, int SLABS, bool KEYS>
__global__ void __launch_bounds__(512, SLABS == 0 ? 1 : (SLABS == 1 ? 3 : 2))
attention_prepare_vec_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, AttnInputs in,
                             const uint32_t *__restrict__ positions, const uint32_t *__restrict__ slot_block,
                             const uint32_t *__restrict__ slot_slot, T *__restrict__ q_out, T *__restrict__ arena, KvLayout kv,
                             uint32_t layer, float *__restrict__ gate) {
  __shared__ float2 red[32];
  pdl_trigger();
  const uint32_t row = blockIdx.x, tid = threadIdx.x, half = in.rope_dims / 2;
  const float *p = partial + (size_t)row * in.ld;
  const uint32_t nq = in.q_heads * in.dim, nk = in.kv_heads * in.dim, nv = KEYS ? 0 : in.kv_heads * in.value_dim, all = nq + nk + nv;
  const uint32_t pos = positions[row], block = slot_block[row], slot = slot_slot[row];
  // gain and angles of the four columns from i on
  auto constants = [&](uint32_t i, float4 &gain, float2 &co, float2 &si) {
    gain = make_float4(1.f, 1.f, 1.f, 1.f), co = make_float2(1.f, 1.f), si = make_float2(0.f, 0.f);
    if (i >= nq + nk) return;
    if (KEYS) {
      if (i < nq) gain = *reinterpret_cast<const float4 *>(in.q_norm + i);
      return;
    }
    if (in.q_norm) gain = *reinterpret_cast<const float4 *>(i < nq ? in.q_norm + i : in.k_norm + (i - nq));
    const uint32_t d = (i < nq ? i : i - nq) % in.dim;
    if (d < in.rope_dims) {
      co = *reinterpret_cast<const float2 *>(in.rope_cos + (size_t)pos * half + d / 2);
      si = *reinterpret_cast<const float2 *>(in.rope_sin + (size_t)pos * half + d / 2);
    }
  };
  constexpr bool kLate = SLABS != 0;
  constexpr int kEarly = kLate ? 1 : GROUPS;
  float4 gain[kEarly];
  float2 co[kEarly], si[kEarly];
  if (!kLate) {
#pragma unroll
    for (int g = 0; g < kEarly; ++g) constants((tid + g * blockDim.x) * 4, gain[g], co[g], si[g]);
  }
  pdl_wait();
  float4 v[GROUPS];
  float sq = 0.f, sk = 0.f;
#pragma unroll
  for (int g = 0; g < GROUPS; ++g) {
    const uint32_t i = (tid + g * blockDim.x) * 4;
    v[g] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (i >= all) continue;
    v[g] = sum_slabs4_most<SLABS>(p + i, splits, split_stride);
    if (KEYS && in.bias) {
      const float4 b = *reinterpret_cast<const float4 *>(in.bias + i);
      v[g] = make_float4(v[g].x + b.x, v[g].y + b.y, v[g].z + b.z, v[g].w + b.w);
    }
    const float s = v[g].x * v[g].x + v[g].y * v[g].y + v[g].z * v[g].z + v[g].w * v[g].w;
    if (i < nq) sq += s;
    else if (i < nq + nk) sk += s;
  }
  if (gate && tid < in.q_heads) gate[(size_t)row * in.q_heads + tid] = sigmoid_f(fold(p + all + tid, splits, split_stride));
  const float2 ss = block_sum2(sq, sk, red);
  const float scale_q = (KEYS || in.q_norm ? 1.0f / sqrtf(ss.x / (float)nq + in.eps) : 1.f) * (KEYS && in.q_factor ? in.q_factor[pos] : 1.f);
  const float scale_k = KEYS || in.q_norm ? 1.0f / sqrtf(ss.y / (float)nk + in.eps) : 1.f;
  if (KEYS && tid < in.kv_heads) *reinterpret_cast<float *>(arena + kv.factor(layer, block, tid, slot)) = scale_k;
#pragma unroll
  for (int g = 0; g < GROUPS; ++g) {
    const uint32_t i = (tid + g * blockDim.x) * 4;
    if (i >= all) continue;
    float4 x = v[g];
    if (KEYS) {
      const int e = kLate ? 0 : g;
      if (kLate) constants(i, gain[e], co[e], si[e]);
      if (i < nq) x = make_float4(x.x * scale_q * gain[e].x, x.y * scale_q * gain[e].y, x.z * scale_q * gain[e].z, x.w * scale_q * gain[e].w);
    } else if (i < nq + nk) {
      const int e = kLate ? 0 : g;
      if (kLate) constants(i, gain[e], co[e], si[e]);
      const float s = i < nq ? scale_q : scale_k;
      x = make_float4(x.x * s * gain[e].x, x.y * s * gain[e].y, x.z * s * gain[e].z, x.w * s * gain[e].w);
      x = make_float4(x.x * co[e].x - x.y * si[e].x, x.y * co[e].x + x.x * si[e].x, x.z * co[e].y - x.w * si[e].y, x.w * co[e].y + x.z * si[e].y);
    }
    if (i < nq) {
      store4<T>(q_out + ((size_t)row * in.q_heads + i / in.dim) * kv.head_dim + i % in.dim, x);
    } else {
      const uint32_t is_v = i >= nq + nk, c = is_v ? i - nq - nk : i - nq, n = is_v ? in.value_dim : in.dim;
      store4<T>(arena + kv.row(layer, block, c / n, is_v, slot) + kv.col(slot, c % n), x);
    }
  }
}

constexpr uint32_t kHeadWarps = 8;

template <int VEC>
__device__ __forceinline__ void load_folded(const float *p, uint32_t splits, size_t stride, float (&v)[VEC]) {
  if (VEC == 4) {
    const float4 x = sum_slabs4(p, splits, stride);
    v[0] = x.x, v[1 % VEC] = x.y, v[2 % VEC] = x.z, v[3 % VEC] = x.w;
  } else {
    v[0] = fold(p, splits, stride);
  }
}
template <typename T, int VEC>
__device__ __forceinline__ void store_values(T *p, const float (&v)[VEC]) {
  if (VEC == 4) store4<T>(p, make_float4(v[0], v[1 % VEC], v[2 % VEC], v[3 % VEC]));
  else p[0] = from_f32<T>(v[0]);
}

// A warp per (row, head of q, k, v or the gate). VEC columns per lane and round: 4 where sizes, strides and rotated halves are multiples
// of 4. A head that rotates passes through shared memory, since its pairs may be any distance apart.
template <typename T, int VEC>
__global__ void __launch_bounds__(kHeadWarps * 32)
attention_prepare_heads_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, AttnInputs in,
                               const uint32_t *__restrict__ positions, const uint32_t *__restrict__ slot_block,
                               const uint32_t *__restrict__ slot_slot, T *__restrict__ q_out, T *__restrict__ arena, KvLayout kv, uint32_t layer,
                               T *__restrict__ value_gate) {
  extern __shared__ __align__(16) float head_values[];  // [kHeadWarps][dim]
  pdl_trigger();
  const uint32_t row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = in.rope_dims / 2;
  const uint32_t nq = in.q_heads * in.dim, nk = in.kv_heads * in.dim, nv = in.kv_heads * in.value_dim;
  const uint32_t pos = positions[row], block = slot_block[row], slot = slot_slot[row];
  const float *cs = in.rope_cos + (size_t)pos * half, *sn = in.rope_sin + (size_t)pos * half;
  const uint32_t first_v = in.q_heads + in.kv_heads, first_gate = first_v + in.kv_heads, heads = first_gate + (value_gate ? in.q_heads : 0);
  float *buf = head_values + warp * in.dim;
  pdl_wait();
  for (uint32_t t = blockIdx.y * kHeadWarps + warp; t < heads; t += gridDim.y * kHeadWarps) {
    if (t >= first_v) {  // values and gates pass straight through
      const bool is_gate = t >= first_gate;
      const uint32_t head = is_gate ? t - first_gate : t - first_v, at = nq + nk + (is_gate ? nv : 0) + head * in.value_dim;
      T *dst = is_gate ? value_gate + ((size_t)row * in.q_heads + head) * in.value_dim : arena + kv.row(layer, block, head, 1, slot);
      for (uint32_t d = lane * VEC; d < in.value_dim; d += 32 * VEC) {
        float v[VEC];
        load_folded<VEC>(partial + (size_t)row * in.ld + at + d, splits, split_stride, v);
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = is_gate ? sigmoid_for<T>(v[i]) : v[i] + (in.bias ? in.bias[at + d + i] : 0.f);
        store_values<T, VEC>(dst + (is_gate ? d : kv.col(slot, d)), v);
      }
      continue;
    }
    const bool is_q = t < in.q_heads;
    const uint32_t head = is_q ? t : t - in.q_heads, at = is_q ? head * in.dim : nq + head * in.dim;
    const float *gain = is_q ? in.q_norm : in.k_norm;
    float ss = 0.f;
    for (uint32_t d = lane * VEC; d < in.dim; d += 32 * VEC) {
      float v[VEC];
      load_folded<VEC>(partial + (size_t)row * in.ld + at + d, splits, split_stride, v);
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        if (in.bias) v[i] += in.bias[at + d + i];
        ss += v[i] * v[i];
        if (gain) v[i] *= gain[d + i];
      }
      store_values<float, VEC>(buf + d, v);
    }
    const float scale = gain ? 1.0f / sqrtf(warp_sum(ss) / (float)in.dim + in.eps) : 1.f;
    __syncwarp();
    T *dst = is_q ? q_out + ((size_t)row * in.q_heads + head) * kv.head_dim : arena + kv.row(layer, block, head, 0, slot);
    for (uint32_t d = lane * VEC; d < in.dim; d += 32 * VEC) {
      float v[VEC];
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        const uint32_t c = d + i;
        v[i] = buf[c];
        if (c < 2 * half) {
          const uint32_t pair = in.halves ? (c < half ? c : c - half) : c >> 1, other = in.halves ? (c < half ? c + half : c - half) : c ^ 1u;
          const bool second = in.halves ? c >= half : c & 1u;
          v[i] = second ? v[i] * cs[pair] + buf[other] * sn[pair] : v[i] * cs[pair] - buf[other] * sn[pair];
        }
        v[i] *= scale;
      }
      store_values<T, VEC>(dst + (is_q ? d : kv.col(slot, d)), v);
    }
    __syncwarp();
  }
}

// The same for heads of at most 128 values (sizes and strides multiples of 4, rotated halves too): a lane holds four columns of each of
// its warp's HEADS heads, all fetched at once, and pairs meet through shuffles. SLABS as above.
template <typename T, int HEADS, int SLABS>
__global__ void __launch_bounds__(kHeadWarps * 32)
attention_prepare_lanes_kernel(const float *__restrict__ partial, uint32_t splits, size_t split_stride, AttnInputs in,
                               const uint32_t *__restrict__ positions, const uint32_t *__restrict__ slot_block,
                               const uint32_t *__restrict__ slot_slot, T *__restrict__ q_out, T *__restrict__ arena, KvLayout kv, uint32_t layer,
                               T *__restrict__ value_gate) {
  pdl_trigger();
  const uint32_t row = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, half = in.rope_dims / 2, d = lane * 4;
  const uint32_t nq = in.q_heads * in.dim, nk = in.kv_heads * in.dim;
  const uint32_t pos = positions[row], block = slot_block[row], slot = slot_slot[row];
  const uint32_t first_v = in.q_heads + in.kv_heads, first_gate = first_v + in.kv_heads, heads = first_gate + (value_gate ? in.q_heads : 0);
  // angles: the first of a pair adds -sin of the other, the second +sin
  const float4 one = make_float4(1.f, 1.f, 1.f, 1.f), zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 co = one, si = zero, gq = one, gk = one;
  uint32_t partner = lane;
  if (d < 2 * half) {
    const uint32_t at = d < half ? d : d - half;
    co = *reinterpret_cast<const float4 *>(in.rope_cos + (size_t)pos * half + at);
    si = *reinterpret_cast<const float4 *>(in.rope_sin + (size_t)pos * half + at);
    if (d < half) si = make_float4(-si.x, -si.y, -si.z, -si.w);
    partner = d < half ? lane + half / 4 : lane - half / 4;
  }
  if (in.q_norm && d < in.dim) {
    gq = *reinterpret_cast<const float4 *>(in.q_norm + d);
    gk = *reinterpret_cast<const float4 *>(in.k_norm + d);
  }
  pdl_wait();
  float4 v[HEADS];
#pragma unroll
  for (int r = 0; r < HEADS; ++r) {
    const uint32_t t = (blockIdx.y * HEADS + r) * kHeadWarps + warp, n = t < first_v ? in.dim : in.value_dim;
    v[r] = zero;
    if (t >= heads || d >= n) continue;
    const uint32_t at = (t < first_v ? t * in.dim : nq + nk + (t - first_v) * in.value_dim) + d;  // gates follow the values
    v[r] = sum_slabs4_most<SLABS>(partial + (size_t)row * in.ld + at, splits, split_stride);
    if (in.bias && t < first_gate) {
      const float4 b = *reinterpret_cast<const float4 *>(in.bias + at);
      v[r] = make_float4(v[r].x + b.x, v[r].y + b.y, v[r].z + b.z, v[r].w + b.w);
    }
  }
#pragma unroll
  for (int r = 0; r < HEADS; ++r) {
    const uint32_t t = (blockIdx.y * HEADS + r) * kHeadWarps + warp;
    if (t >= heads) continue;
    float4 x = v[r];
    if (t >= first_gate) {
      x = make_float4(sigmoid_for<T>(x.x), sigmoid_for<T>(x.y), sigmoid_for<T>(x.z), sigmoid_for<T>(x.w));
      if (d < in.value_dim) store4<T>(value_gate + ((size_t)row * in.q_heads + (t - first_gate)) * in.value_dim + d, x);
      continue;
    }
    if (t >= first_v) {
      if (d < in.value_dim) store4<T>(arena + kv.row(layer, block, t - first_v, 1, slot) + kv.col(slot, d), x);
      continue;
    }
    const bool is_q = t < in.q_heads;
    if (in.q_norm) {
      const float s = 1.0f / sqrtf(warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w) / (float)in.dim + in.eps);
      const float4 g = is_q ? gq : gk;
      x = make_float4(x.x * s * g.x, x.y * s * g.y, x.z * s * g.z, x.w * s * g.w);
    }
    const float4 o = make_float4(__shfl_sync(0xffffffffu, x.x, partner), __shfl_sync(0xffffffffu, x.y, partner),
                                 __shfl_sync(0xffffffffu, x.z, partner), __shfl_sync(0xffffffffu, x.w, partner));
    x = make_float4(x.x * co.x + o.x * si.x, x.y * co.y + o.y * si.y, x.z * co.z + o.z * si.z, x.w * co.w + o.w * si.w);
    if (d >= in.dim) continue;
    if (is_q) store4<T>(q_out + ((size_t)row * in.q_heads + t) * kv.head_dim + d, x);
    else store4<T>(arena + kv.row(layer, block, t - in.q_heads, 0, slot) + kv.col(slot, d), x);
  }
}

template <typename T>
__global__ void arena_rows_kernel(const T *__restrict__ arena, KvLayout kv, uint32_t dim, uint32_t value_dim, float *__restrict__ out) {
  const bool factors = kv.factor_elems > 0;  // in the place of V rows: one value per slot
  if (factors) value_dim = 1;
  const size_t tokens = (size_t)kv.num_blocks * kv.num_kv_heads * kv.block_size, keys = tokens * dim, all = keys + tokens * value_dim;
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < all; i += (size_t)gridDim.x * blockDim.x) {
    const uint32_t is_v = i >= keys, n = is_v ? value_dim : dim;
    const size_t j = is_v ? i - keys : i, t = j / n;
    const uint32_t slot = t % kv.block_size, head = t / kv.block_size % kv.num_kv_heads;
    const uint32_t block = (uint32_t)(t / kv.block_size / kv.num_kv_heads);
    out[i] = factors && is_v ? *reinterpret_cast<const float *>(arena + kv.factor(0, block, head, slot))
                             : to_f32<T>(arena[kv.row(0, block, head, is_v, slot) + kv.col(slot, j % n)]);
  }
}

template <typename T>
__global__ void fill_factors_kernel(T *__restrict__ arena, KvLayout kv, float value) {
  const size_t tokens = (size_t)kv.num_blocks * kv.num_kv_heads * kv.block_size;
  for (size_t t = (size_t)blockIdx.x * blockDim.x + threadIdx.x; t < tokens; t += (size_t)gridDim.x * blockDim.x)
    *reinterpret_cast<float *>(arena + kv.factor(0, (uint32_t)(t / kv.block_size / kv.num_kv_heads), t / kv.block_size % kv.num_kv_heads, t % kv.block_size)) = value;
}

inline int after_launch(const char *stage) {
  count_launch();
  ORION_CUDA_CHECK(stage, cudaGetLastError());
  return ORION_OK;
}

template <typename T, int GROUPS, int SLABS, bool KEYS>
int launch_vec(const float *partial, uint32_t splits, size_t split_stride, AttnInputs in, const uint32_t *positions, const uint32_t *slot_block,
               const uint32_t *slot_slot, T *q_out, T *arena, KvLayout kv, uint32_t layer, float *gate, uint32_t rows, uint32_t threads,
               cudaStream_t stream) {
  ORION_CUDA_CHECK("attention_prepare", launch_pdl(attention_prepare_vec_kernel<T, GROUPS, SLABS, KEYS>, dim3(rows), dim3(threads), 0, stream, partial, splits,
                                                   split_stride, in, positions, slot_block, slot_slot, q_out, arena, kv, layer, gate));
  return after_launch("attention_prepare");
}

// The variant for this many rounds and slabs; null if there is none.
template <typename T, bool KEYS>
auto vec_variant(uint32_t rounds, int slabs) {
  auto pick = [&](auto none, auto one, auto four) { return slabs == 1 ? one : (slabs == 4 ? four : none); };
  return rounds == 1   ? pick(launch_vec<T, 1, 0, KEYS>, launch_vec<T, 1, 1, KEYS>, launch_vec<T, 1, 4, KEYS>)
         : rounds == 2 ? pick(launch_vec<T, 2, 0, KEYS>, launch_vec<T, 2, 1, KEYS>, launch_vec<T, 2, 4, KEYS>)
         : rounds == 4 ? pick(launch_vec<T, 4, 0, KEYS>, launch_vec<T, 4, 1, KEYS>, launch_vec<T, 4, 4, KEYS>)
                       : launch_vec<T, 8, 0, KEYS>;
}

}  // namespace

template <typename T>
int launch_attention_prepare(const float *partial, uint32_t splits, size_t split_stride, AttnInputs in, const uint32_t *positions,
                             const uint32_t *slot_block, const uint32_t *slot_slot, T *q_out, T *arena, KvLayout kv, uint32_t layer,
                             float *gate, uint32_t rows, cudaStream_t stream, T *value_gate) {
  if (rows == 0) return ORION_OK;
  if (in.per_head) {
    if (gate) return set_error(ORION_ERR_INTERNAL, "a gate per head is not built for this layout");
    const bool vec = in.dim % 4 == 0 && in.value_dim % 4 == 0 && in.rope_dims % 4 == 0 && in.ld % 4 == 0 && split_stride % 4 == 0 &&
                     kv.head_dim % 4 == 0 && kv.v_dim() % 4 == 0;
    const uint32_t heads = 2 * in.kv_heads + in.q_heads * (value_gate ? 2 : 1);
    if (vec && in.dim <= 128 && in.value_dim <= 128 && in.halves && in.rope_dims % 8 == 0) {
      const int slabs = slab_variant(rows, splits);
      const uint32_t each = slabs == 0 || rows < 296 ? 1 : (slabs == 4 ? 2 : 5);  // heads per warp
      auto kernel = each == 1 ? attention_prepare_lanes_kernel<T, 1, 0> : (each == 2 ? attention_prepare_lanes_kernel<T, 2, 4> : attention_prepare_lanes_kernel<T, 5, 1>);
      ORION_CUDA_CHECK("attention_prepare", launch_pdl(kernel, dim3(rows, (heads + each * kHeadWarps - 1) / (each * kHeadWarps)), dim3(kHeadWarps * 32), 0,
                                                       stream, partial, splits, split_stride, in, positions, slot_block, slot_slot, q_out, arena, kv,
                                                       layer, value_gate));
      return after_launch("attention_prepare");
    }
    const uint32_t most = (heads + kHeadWarps - 1) / kHeadWarps;
    // decode batches: a warp per head; prompts: a CTA per row
    const uint32_t split = rows >= 1024 ? 1 : (most < 1024 / rows + 1 ? most : 1024 / rows + 1);
    const size_t smem = (size_t)kHeadWarps * in.dim * sizeof(float);
    if (smem > 48 * 1024) return set_error(ORION_ERR_INTERNAL, "query and key heads of %u values are not supported", in.dim);
    ORION_CUDA_CHECK("attention_prepare", launch_pdl(vec ? attention_prepare_heads_kernel<T, 4> : attention_prepare_heads_kernel<T, 1>, dim3(rows, split),
                                                     dim3(kHeadWarps * 32), smem, stream, partial, splits, split_stride, in, positions, slot_block,
                                                     slot_slot, q_out, arena, kv, layer, value_gate));
    return after_launch("attention_prepare");
  }
  if (in.halves || value_gate || (in.bias && !in.keys_as_values))
    return set_error(ORION_ERR_INTERNAL, "rotated halves, biases and gates per value come with norms per head");
  if (in.keys_as_values && (!in.q_norm || in.rope_dims || gate || kv.factor_elems * sizeof(T) != sizeof(float) || in.value_dim != in.dim))
    return set_error(ORION_ERR_INTERNAL, "keys as values come with norms, without rotation and gates, and one set of rows");
  if ((in.q_norm == nullptr) != (in.k_norm == nullptr)) return set_error(ORION_ERR_INTERNAL, "query and key norms come together");
  const uint32_t groups = (in.q_heads * in.dim + in.kv_heads * (in.dim + (in.keys_as_values ? 0 : in.value_dim))) / 4;
  const uint32_t rounds = groups <= 256 ? 1 : (groups <= 1024 ? 2 : (groups <= 2048 ? 4 : 8));
  const uint32_t threads = ((groups + rounds - 1) / rounds + 31) / 32 * 32;
  if (in.dim % 4 == 0 && in.value_dim % 4 == 0 && in.rope_dims % 4 == 0 && in.ld % 4 == 0 && split_stride % 4 == 0 && kv.head_dim % 4 == 0 &&
      kv.v_dim() % 4 == 0 && threads <= 512 && in.q_heads <= threads && in.kv_heads <= threads) {
    const int slabs = slab_variant(rows, splits);
    auto run = in.keys_as_values ? vec_variant<T, true>(rounds, slabs) : vec_variant<T, false>(rounds, slabs);
    return run(partial, splits, split_stride, in, positions, slot_block, slot_slot, q_out, arena, kv, layer, gate, rows, threads, stream);
  }
  ORION_CUDA_CHECK("attention_prepare", launch_pdl(attention_prepare_kernel<T>, dim3(rows), dim3(256), 0, stream, partial, splits, split_stride, in,
                                                   positions, slot_block, slot_slot, q_out, arena, kv, layer, gate));
  return after_launch("attention_prepare");
}

template <typename T>
int launch_arena_rows(const T *arena, KvLayout kv, uint32_t dim, uint32_t value_dim, float *out, cudaStream_t stream) {
  arena_rows_kernel<T><<<148 * 8, 256, 0, stream>>>(arena, kv, dim, value_dim, out);
  return after_launch("arena_rows");
}

template <typename T>
int launch_fill_factors(T *arena, KvLayout kv, float value, cudaStream_t stream) {
  fill_factors_kernel<T><<<148 * 8, 256, 0, stream>>>(arena, kv, value);
  return after_launch("fill_factors");
}

#define ORION_INSTANTIATE(T)                                                                                                            \
  template int launch_attention_prepare<T>(const float *, uint32_t, size_t, AttnInputs, const uint32_t *, const uint32_t *, const uint32_t *, \
                                           T *, T *, KvLayout, uint32_t, float *, uint32_t, cudaStream_t, T *);                         \
  template int launch_arena_rows<T>(const T *, KvLayout, uint32_t, uint32_t, float *, cudaStream_t);                                   \
  template int launch_fill_factors<T>(T *, KvLayout, float, cudaStream_t);
ORION_INSTANTIATE(float)
ORION_INSTANTIATE(bf16)

}  // namespace orion
