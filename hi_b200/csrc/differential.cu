// Differential attention's last step, for the attention kernels that leave their rows as split partials: merge the
// splits of both maps of a head, subtract, norm over the head's values, gate.
//
//   a_m = sum_s acc_s e^{m_s - m} / sum_s l_s e^{m_s - m}        for map m of the head (heads 2h and 2h + 1 of the partials)
//   o = a_1 - lambda a_2;   o <- o rsqrt(mean over vdim of o^2 + eps) mul;   out = o * sigmoid(gate)
//
// and gate_rows, out = o * sigmoid(gate) alone, for attention without the second map.
#include "api.h"
#include "common.cuh"

namespace {

// One block per (row, head), half its threads per map. `rows` maps a row of the partials to a row of `out` and of the
// gate (null: the same).
template <typename T>
__global__ void __launch_bounds__(256) diff_merge_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                  const long long* __restrict__ rows, const T* __restrict__ gate, long long gate_stride,
                                  T* __restrict__ out, int heads, int hd, int vdim, int splits, float lambda, float eps,
                                  float mul) {
  extern __shared__ float sm_d[];              // [2][splits] weights, [2] 1 / sum, [2][vdim] rows, 33 scratch
  float* wgt = sm_d;
  float* inv_l = wgt + 2 * splits;
  float* val = inv_l + 2;
  float* scratch = val + 2 * vdim;
  const int h = blockIdx.y;
  const size_t r = blockIdx.x;
  const size_t dst = rows ? (size_t)rows[r] : r;
  const int half = blockDim.x / 2;             // whole warps
  const int mp = threadIdx.x / half, tid = threadIdx.x % half;
  const float* acc = part_acc + ((r * heads + h) * 2 + mp) * (size_t)splits * hd;
  // partial rows of the first splits are asked for before the weights are worked out; a split past the token's range
  // has an unwritten row, which may be loaded but must not enter the sum (its weight is 0)
  constexpr int AHEAD = 8;
  float ahead[AHEAD];
  if (tid < vdim) {
#pragma unroll
    for (int s = 0; s < AHEAD; ++s)
      if (s < splits) ahead[s] = acc[(size_t)s * hd + tid];
  }
  float g0 = 0.f;
  if (gate && tid < vdim) g0 = hb::to_f32(gate[dst * gate_stride + (size_t)h * vdim + tid]);
  if (threadIdx.x % half < 32) {               // the first warp of each half: its map's weights
    const float* ml = part_ml + ((r * heads + h) * 2 + mp) * (size_t)splits * 2;
    float m = -INFINITY;
    for (int s = tid; s < splits; s += 32) m = fmaxf(m, ml[2 * s]);
    m = hb::warp_max(m);
    float l = 0.f;
    for (int s = tid; s < splits; s += 32) {
      const float ms = ml[2 * s];
      const float e = ms == -INFINITY ? 0.f : expf(ms - m);
      wgt[mp * splits + s] = e;
      l += ml[2 * s + 1] * e;
    }
    l = hb::warp_sum(l);
    if (tid == 0) inv_l[mp] = l > 0.f ? 1.f / l : 0.f;
  }
  __syncthreads();
  for (int d = tid; d < vdim; d += half) {
    float o = 0.f;
    int s = 0;
    if (d == tid) {
#pragma unroll
      for (int q = 0; q < AHEAD; ++q)
        if (q < splits) {
          const float w = wgt[mp * splits + q];
          if (w != 0.f) o += ahead[q] * w;
        }
      s = min(splits, AHEAD);
    }
#pragma unroll 8
    for (; s < splits; ++s) {
      const float w = wgt[mp * splits + s];
      if (w != 0.f) o += acc[(size_t)s * hd + d] * w;
    }
    val[mp * vdim + d] = o * inv_l[mp];
  }
  __syncthreads();
  float ss = 0.f;
  for (int d = threadIdx.x; d < vdim; d += blockDim.x) {
    const float o = val[d] - lambda * val[vdim + d];
    ss += o * o;
  }
  ss = hb::block_sum(ss, scratch);
  const float f = rsqrtf(ss / (float)vdim + eps) * mul;
  for (int d = threadIdx.x; d < vdim; d += blockDim.x) {
    float o = (val[d] - lambda * val[vdim + d]) * f;
    if (gate) {
      const float g = d == tid ? g0 : hb::to_f32(gate[dst * gate_stride + (size_t)h * vdim + d]);
      o /= 1.f + expf(-g);
    }
    out[(dst * heads + h) * vdim + d] = hb::from_f32<T>(o);
  }
}

// One split (portions of prompts): a warp per (row, head), four channels a lane and pass; vdim % 4 == 0, vdim <= 512.
template <typename T>
__global__ void __launch_bounds__(128) diff_rows_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                 const T* __restrict__ gate, long long gate_stride, T* __restrict__ out, long long n_rows,
                                 int heads, int hd, int vdim, float lambda, float eps, float mul) {
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= n_rows * heads) return;
  const long long r = w / heads;
  const int h = (int)(w - r * heads);
  const float* a1 = part_acc + (size_t)w * 2 * hd;
  const float* a2 = a1 + hd;
  const float l1 = part_ml[w * 4 + 1], l2 = part_ml[w * 4 + 3];
  const float f1 = l1 > 0.f ? 1.f / l1 : 0.f, f2 = l2 > 0.f ? lambda / l2 : 0.f;
  constexpr int PASSES = 4;
  float4 v[PASSES];
  float ss = 0.f;
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int d = (p * 32 + lane) * 4;
    if (d < vdim) {
      const float4 x = *reinterpret_cast<const float4*>(a1 + d), y = *reinterpret_cast<const float4*>(a2 + d);
      v[p] = make_float4(x.x * f1 - y.x * f2, x.y * f1 - y.y * f2, x.z * f1 - y.z * f2, x.w * f1 - y.w * f2);
      ss += v[p].x * v[p].x + v[p].y * v[p].y + v[p].z * v[p].z + v[p].w * v[p].w;
    }
  }
  ss = hb::warp_sum(ss);
  const float f = rsqrtf(ss / (float)vdim + eps) * mul;
#pragma unroll
  for (int p = 0; p < PASSES; ++p) {
    const int d = (p * 32 + lane) * 4;
    if (d < vdim) {
      float o[4] = {v[p].x * f, v[p].y * f, v[p].z * f, v[p].w * f};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (gate) o[e] /= 1.f + expf(-hb::to_f32(gate[r * gate_stride + (size_t)h * vdim + d + e]));
        out[(size_t)w * vdim + d + e] = hb::from_f32<T>(o[e]);
      }
    }
  }
}

template <typename T>
__global__ void gate_rows_kernel(const T* __restrict__ o, long long o_stride, const T* __restrict__ gate, long long gate_stride,
                                 T* __restrict__ out, long long rows, int heads, int hd, int vdim) {
  const long long width = (long long)heads * vdim, total = rows * width;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / width;
    const int c = (int)(i - r * width), h = c / vdim, d = c - h * vdim;
    const float x = hb::to_f32(o[r * o_stride + (size_t)h * hd + d]);
    out[i] = hb::from_f32<T>(x / (1.f + expf(-hb::to_f32(gate[r * gate_stride + c]))));
  }
}

__device__ __forceinline__ void put8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void put8(__nv_bfloat16* p, const float (&v)[8]) {
  alignas(16) __nv_bfloat162 h[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = *reinterpret_cast<uint4*>(h);
}

// The same, eight neighbouring values a thread: head sizes and strides multiples of eight, rows on 16 bytes. Grid
// (blocks over a row's eights, rows).
template <typename T>
__global__ void gate_rows8_kernel(const T* __restrict__ o, long long o_stride, const T* __restrict__ gate, long long gate_stride,
                                  T* __restrict__ out, int heads, int hd, int vdim) {
  const size_t r = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  if (c >= heads * vdim) return;
  const int h = c / vdim;
  float x[8], g[8];
  hb::load8(o + r * o_stride + (size_t)h * hd + (c - h * vdim), x);
  hb::load8(gate + r * gate_stride + c, g);
#pragma unroll
  for (int i = 0; i < 8; ++i) x[i] /= 1.f + expf(-g[i]);
  put8(out + r * (size_t)heads * vdim + c, x);
}

}  // namespace

// part_acc [n_rows][2 * heads][splits][hd], part_ml [n_rows][2 * heads][splits][2] -> out [.][heads][vdim]
extern "C" int hb_diff_merge(const float* part_acc, const float* part_ml, const long long* rows, const void* gate,
                             long long gate_stride, void* out, int dtype, int n_rows, int heads, int hd, int vdim, int splits,
                             float lambda, float eps, float mul, cudaStream_t stream) {
  if (!part_acc || !part_ml || !out || n_rows < 0 || heads <= 0 || heads > 65535 || hd <= 0 || vdim <= 0 || vdim > hd || splits < 1)
    return HB_ERR_BAD_ARG;
  if (dtype != HB_DTYPE_F32 && dtype != HB_DTYPE_BF16) return HB_ERR_BAD_ARG;
  if (n_rows == 0) return HB_OK;
  if (splits == 1 && !rows && vdim % 4 == 0 && hd % 4 == 0 && vdim <= 512) {
    const long long warps = (long long)n_rows * heads, blocks = (warps + 3) / 4;
    if (blocks > 0x7fffffffLL) return HB_ERR_UNSUPPORTED;
    if (dtype == HB_DTYPE_F32)
      diff_rows_kernel<float><<<(int)blocks, 128, 0, stream>>>(part_acc, part_ml, (const float*)gate, gate_stride, (float*)out,
                                                               n_rows, heads, hd, vdim, lambda, eps, mul);
    else
      diff_rows_kernel<__nv_bfloat16><<<(int)blocks, 128, 0, stream>>>(
          part_acc, part_ml, (const __nv_bfloat16*)gate, gate_stride, (__nv_bfloat16*)out, n_rows, heads, hd, vdim, lambda, eps, mul);
    HB_LAUNCH_CHECK();
    return HB_OK;
  }
  const size_t smem = (size_t)(2 * splits + 2 + 2 * vdim + 33) * sizeof(float);
  if (smem > 48 * 1024) return HB_ERR_UNSUPPORTED;
  const dim3 grid(n_rows, heads);
  const int threads = vdim <= 64 ? 128 : 256;
  if (dtype == HB_DTYPE_F32)
    diff_merge_kernel<float><<<grid, threads, smem, stream>>>(part_acc, part_ml, rows, (const float*)gate, gate_stride, (float*)out,
                                                              heads, hd, vdim, splits, lambda, eps, mul);
  else
    diff_merge_kernel<__nv_bfloat16><<<grid, threads, smem, stream>>>(
        part_acc, part_ml, rows, (const __nv_bfloat16*)gate, gate_stride, (__nv_bfloat16*)out, heads, hd, vdim, splits, lambda, eps, mul);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

// out [rows, heads * vdim] = o * sigmoid(gate); row r of o at o + r * o_stride, its heads hd apart
extern "C" int hb_gate_rows(const void* o, long long o_stride, const void* gate, long long gate_stride, void* out, int dtype,
                            long long rows, int heads, int hd, int vdim, cudaStream_t stream) {
  if (!o || !gate || !out || rows < 0 || heads <= 0 || hd <= 0 || vdim <= 0 || vdim > hd) return HB_ERR_BAD_ARG;
  if (rows == 0) return HB_OK;
  const bool wide = hd % 8 == 0 && vdim % 8 == 0 && o_stride % 8 == 0 && gate_stride % 8 == 0 && rows <= 65535 &&
                    (reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(gate) | reinterpret_cast<uintptr_t>(out)) % 16 == 0;
  if (wide && (dtype == HB_DTYPE_F32 || dtype == HB_DTYPE_BF16)) {
    const int eights = heads * vdim / 8, threads = eights >= 256 ? 256 : (eights + 31) / 32 * 32;
    const dim3 grid((eights + threads - 1) / threads, (unsigned)rows);
    if (dtype == HB_DTYPE_F32)
      gate_rows8_kernel<float><<<grid, threads, 0, stream>>>((const float*)o, o_stride, (const float*)gate, gate_stride, (float*)out, heads, hd, vdim);
    else
      gate_rows8_kernel<__nv_bfloat16><<<grid, threads, 0, stream>>>((const __nv_bfloat16*)o, o_stride, (const __nv_bfloat16*)gate, gate_stride,
                                                                     (__nv_bfloat16*)out, heads, hd, vdim);
    HB_LAUNCH_CHECK();
    return HB_OK;
  }
  const long long want = (rows * heads * vdim + 255) / 256;
  const int blocks = (int)(want < 148 * 16 ? want : 148 * 16);
  if (dtype == HB_DTYPE_F32)
    gate_rows_kernel<float><<<blocks, 256, 0, stream>>>((const float*)o, o_stride, (const float*)gate, gate_stride, (float*)out, rows, heads, hd, vdim);
  else if (dtype == HB_DTYPE_BF16)
    gate_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, stream>>>((const __nv_bfloat16*)o, o_stride, (const __nv_bfloat16*)gate, gate_stride,
                                                                (__nv_bfloat16*)out, rows, heads, hd, vdim);
  else
    return HB_ERR_BAD_ARG;
  HB_LAUNCH_CHECK();
  return HB_OK;
}
