// Boundary of a block that norms what a sub-layer read AND what it returned:
//
//   y = delta + delta2 + sum_j routed[slot_j] * weight_j       the sub-layer's open result (any part absent)
//   x <- x + y rsqrt(mean(y^2) + eps_y) w_y                     the stream, float32, in place
//   h = x rsqrt(mean(x^2) + eps) w                              the next sub-layer's input (w null: h = x, where y is given)
//
// One kernel a boundary: the stream is read and written once. With `row_map` only those rows are taken and the stream
// is left as it is (the rows whose logits are wanted). Norm weights are float32 as they act (a weight stored around
// zero already has its 1); statistics and sums are float32.
#include "api.h"
#include "common.cuh"

namespace {

struct SandwichArgs {
  float* x;
  const void* delta;
  int delta_dtype;
  const void* delta2;
  int delta2_dtype;
  const float* routed;
  const int* slot_of_entry;
  const float* routed_weight;
  int top_k;
  const float* w_y;
  float eps_y;
  const float* w;
  float eps;
  void* y;
  int y_dtype;
  float* y_f32;
  const int* row_map;
  int hidden;
};

__device__ __forceinline__ float ld1(const void* p, int dtype, size_t i) {
  return dtype == HB_DTYPE_F32 ? reinterpret_cast<const float*>(p)[i] : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
}
__device__ __forceinline__ float4 ld4(const void* p, int dtype, size_t i) {
  if (dtype == HB_DTYPE_F32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
  return make_float4(__uint_as_float(raw.x << 16), __uint_as_float(raw.x & 0xffff0000u),
                     __uint_as_float(raw.y << 16), __uint_as_float(raw.y & 0xffff0000u));
}
__device__ __forceinline__ void st4(void* p, int dtype, size_t i, float4 v) {
  if (dtype == HB_DTYPE_F32) {
    *reinterpret_cast<float4*>(reinterpret_cast<float*>(p) + i) = v;
  } else {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p) + i) =
        make_uint2(*reinterpret_cast<unsigned*>(&a), *reinterpret_cast<unsigned*>(&b));
  }
}
__device__ __forceinline__ float dot4(float4 a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }

// Any width: the row lives in shared memory.
__global__ void sandwich_kernel(const SandwichArgs a) {
  __shared__ float scratch[33];
  extern __shared__ float row_s[];             // hidden floats
  const int r = blockIdx.x;
  const size_t src = a.row_map ? (size_t)a.row_map[r] : (size_t)r;
  float ss = 0.f;
  for (int j = threadIdx.x; j < a.hidden; j += blockDim.x) {
    float s = 0.f;
    if (a.delta) s += ld1(a.delta, a.delta_dtype, src * a.hidden + j);
    if (a.delta2) s += ld1(a.delta2, a.delta2_dtype, src * a.hidden + j);
    if (a.routed)
      for (int q = 0; q < a.top_k; ++q)
        s += a.routed[(size_t)a.slot_of_entry[src * a.top_k + q] * a.hidden + j] *
             (a.routed_weight ? a.routed_weight[src * a.top_k + q] : 1.f);
    row_s[j] = s;
    ss += s * s;
  }
  const float inv_y = rsqrtf(hb::block_sum(ss, scratch) / (float)a.hidden + a.eps_y);
  ss = 0.f;
  for (int j = threadIdx.x; j < a.hidden; j += blockDim.x) {
    const float s = a.x[src * a.hidden + j] + row_s[j] * inv_y * a.w_y[j];
    if (!a.row_map) a.x[src * a.hidden + j] = s;
    row_s[j] = s;
    ss += s * s;
    if (!a.w && a.y) {
      if (a.y_dtype == HB_DTYPE_F32) reinterpret_cast<float*>(a.y)[src * a.hidden + j] = s;
      else reinterpret_cast<__nv_bfloat16*>(a.y)[src * a.hidden + j] = __float2bfloat16_rn(s);
    }
  }
  if (!a.w) return;
  const float inv = rsqrtf(hb::block_sum(ss, scratch) / (float)a.hidden + a.eps);
  for (int j = threadIdx.x; j < a.hidden; j += blockDim.x) {
    const float o = row_s[j] * inv * a.w[j];
    if (a.y_dtype == HB_DTYPE_F32) reinterpret_cast<float*>(a.y)[(size_t)r * a.hidden + j] = o;
    else reinterpret_cast<__nv_bfloat16*>(a.y)[(size_t)r * a.hidden + j] = __float2bfloat16_rn(o);
    if (a.y_f32) a.y_f32[(size_t)r * a.hidden + j] = o;
  }
}

// hidden % 4 == 0 and hidden <= 4 * blockDim * NG: four columns a thread and group, the row in registers, every load
// asked for before the first use.
template <int NG>
__global__ void __launch_bounds__(512) sandwich_vec_kernel(const SandwichArgs a) {
  __shared__ float scratch[33];
  const int r = blockIdx.x;
  const size_t src = a.row_map ? (size_t)a.row_map[r] : (size_t)r;
  int slots[8];
  float factor[8];
#pragma unroll
  for (int j = 0; j < 8; ++j)
    if (a.routed && j < a.top_k) {
      slots[j] = a.slot_of_entry[src * a.top_k + j];
      factor[j] = a.routed_weight ? a.routed_weight[src * a.top_k + j] : 1.f;
    }
  float4 v[NG], xv[NG], wy[NG], wv[NG];
  float ss = 0.f;
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    const int idx = (threadIdx.x + g * blockDim.x) * 4;
    if (idx < a.hidden) {
      xv[g] = *reinterpret_cast<const float4*>(a.x + src * a.hidden + idx);
      wy[g] = *reinterpret_cast<const float4*>(a.w_y + idx);
      wv[g] = a.w ? *reinterpret_cast<const float4*>(a.w + idx) : make_float4(0.f, 0.f, 0.f, 0.f);
      float4 s = a.delta ? ld4(a.delta, a.delta_dtype, src * a.hidden + idx) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (a.delta2) {
        const float4 d = ld4(a.delta2, a.delta2_dtype, src * a.hidden + idx);
        s.x += d.x; s.y += d.y; s.z += d.z; s.w += d.w;
      }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (a.routed && j < a.top_k) {
          const float4 d = *reinterpret_cast<const float4*>(a.routed + (size_t)slots[j] * a.hidden + idx);
          s.x += d.x * factor[j]; s.y += d.y * factor[j]; s.z += d.z * factor[j]; s.w += d.w * factor[j];
        }
      v[g] = s;
      ss += dot4(s);
    }
  }
  const float inv_y = rsqrtf(hb::block_sum(ss, scratch) / (float)a.hidden + a.eps_y);
  ss = 0.f;
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    const int idx = (threadIdx.x + g * blockDim.x) * 4;
    if (idx < a.hidden) {
      float4 s = v[g];
      s = make_float4(xv[g].x + s.x * inv_y * wy[g].x, xv[g].y + s.y * inv_y * wy[g].y, xv[g].z + s.z * inv_y * wy[g].z,
                      xv[g].w + s.w * inv_y * wy[g].w);
      if (!a.row_map) *reinterpret_cast<float4*>(a.x + src * a.hidden + idx) = s;
      if (!a.w && a.y) st4(a.y, a.y_dtype, src * a.hidden + idx, s);
      v[g] = s;
      ss += dot4(s);
    }
  }
  if (!a.w) return;
  const float inv = rsqrtf(hb::block_sum(ss, scratch) / (float)a.hidden + a.eps);
#pragma unroll
  for (int g = 0; g < NG; ++g) {
    const int idx = (threadIdx.x + g * blockDim.x) * 4;
    if (idx < a.hidden) {
      const float4 o = make_float4(v[g].x * inv * wv[g].x, v[g].y * inv * wv[g].y, v[g].z * inv * wv[g].z, v[g].w * inv * wv[g].w);
      st4(a.y, a.y_dtype, (size_t)r * a.hidden + idx, o);
      if (a.y_f32) *reinterpret_cast<float4*>(a.y_f32 + (size_t)r * a.hidden + idx) = o;
    }
  }
}

bool known(int d) { return d == HB_DTYPE_F32 || d == HB_DTYPE_BF16; }

}  // namespace

extern "C" int hb_sandwich_step(float* x, const void* delta, int delta_dtype, const void* delta2, int delta2_dtype,
                                const float* routed, const int* slot_of_entry, const float* routed_weight, int top_k,
                                const float* w_y, float eps_y, const float* w, float eps, void* y, int y_dtype, float* y_f32,
                                const int* row_map, int rows, int hidden, cudaStream_t stream) {
  if (!x || !w_y || rows < 0 || hidden <= 0 || (delta && !known(delta_dtype)) || (delta2 && !known(delta2_dtype)) ||
      (w && !y) || (y && !known(y_dtype)) || (!w && row_map))
    return HB_ERR_BAD_ARG;
  if (routed && (!slot_of_entry || top_k < 1 || top_k > 8)) return HB_ERR_BAD_ARG;
  if (rows == 0) return HB_OK;
  SandwichArgs a{x, delta, delta_dtype, delta2, delta2_dtype, routed, slot_of_entry, routed_weight, top_k, w_y, eps_y,
                 w, eps, y, y_dtype, y_f32, row_map, hidden};
  if (hidden % 4 == 0 && hidden <= 4 * 512 * 4) {
    const int groups = hidden / 4;
    const int threads = groups >= 512 ? 512 : ((groups + 31) / 32) * 32;
    const int ng = (groups + threads - 1) / threads;
    if (ng <= 1) sandwich_vec_kernel<1><<<rows, threads, 0, stream>>>(a);
    else if (ng <= 2) sandwich_vec_kernel<2><<<rows, threads, 0, stream>>>(a);
    else sandwich_vec_kernel<4><<<rows, threads, 0, stream>>>(a);
    HB_LAUNCH_CHECK();
    return HB_OK;
  }
  const size_t smem = (size_t)hidden * sizeof(float);
  if (smem > 200 * 1024) return HB_ERR_UNSUPPORTED;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(sandwich_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  sandwich_kernel<<<rows, hidden >= 2048 ? 512 : 256, smem, stream>>>(a);
  HB_LAUNCH_CHECK();
  return HB_OK;
}
