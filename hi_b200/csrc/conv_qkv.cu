// After the fused q/k/v projection of an attention layer whose projected channels pass a short causal convolution
// over time: convolution, RMS norm of q and k per head, rotation, and the append of k and v to the paged cache.
//
//   y[t, c] = sum_j taps[c, j] * u[t - (K-1) + j, c]      rows before the portion's first token come from the request's
//                                                         state ([K-1, channels] float32, zero at its start)
//   q, k:  x <- x rsqrt(mean over dim of x^2 + eps) * w   (w [dim] float32, shared by all heads)
//   rotation of the first 2 * rot_pairs dims (general kernel)
//
// Rows of the projection are [q: heads * maps * dim | k: kv_heads * maps * dim | v: kv_heads * vdim | ...], without
// padding. With maps == 2 (differential attention) a head has two query vectors and a kv head two key vectors over one
// value: the key row of a kv head is [map 1 | map 2 | zeros], and query vector (head, map) fills only its own map's
// place of a row of q_out, zeros elsewhere, so the dot product over the whole row is the map's own. A value row is
// [vdim | zeros]. All arithmetic is float32; what is stored is rounded once.
#include "api.h"
#include "common.cuh"

namespace {

struct ConvArgs {
  const void* proj;
  long long ld;                  // elements between rows of proj
  const float* taps;             // [K][channels], or null (K == 1: no convolution)
  float* state;                  // [slots][state_stride], the K - 1 rows of a request at conv_off
  long long state_stride, conv_off;
  const float* q_w;
  const float* k_w;              // [dim] or null
  const float* inv_freq;         // [rot_pairs] or null
  int rot_pairs, interleaved;
  float rot_mul, eps;
  int norm, write_kv, fuse_tail, K;
  const int* positions;
  const int* seq_of_token;
  const int* cu_seqlens;
  const int* slots;
  const int* block_table;
  int table_stride, page_size;
  void* q_out;                   // [n_tokens][heads * maps][hd]
  void* k_pages;
  void* v_pages;                 // [pages][kv_heads][page_size][hd]
  int n_tokens, heads, kv_heads, maps, dim, vdim, hd;
};

__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 pack;
  uint32_t* w = reinterpret_cast<uint32_t*>(&pack);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    w[i] = *reinterpret_cast<uint32_t*>(&h);
  }
  *reinterpret_cast<uint4*>(p) = pack;
}

// 8 consecutive elements as they lie in memory
template <typename T> struct Raw8 { uint4 w[sizeof(T) / 2]; };
template <typename T> __device__ __forceinline__ Raw8<T> raw8(const T* p) {
  Raw8<T> r;
#pragma unroll
  for (int i = 0; i < (int)(sizeof(T) / 2); ++i) r.w[i] = reinterpret_cast<const uint4*>(p)[i];
  return r;
}
__device__ __forceinline__ float element(const Raw8<float>& r, int e) {
  const uint4 q = r.w[e / 4];
  return __uint_as_float(e % 4 == 0 ? q.x : e % 4 == 1 ? q.y : e % 4 == 2 ? q.z : q.w);
}
__device__ __forceinline__ float element(const Raw8<__nv_bfloat16>& r, int e) {
  const uint4 q = r.w[0];
  const uint32_t w = e / 2 == 0 ? q.x : e / 2 == 1 ? q.y : e / 2 == 2 ? q.z : q.w;
  return __uint_as_float(e % 2 ? w & 0xffff0000u : w << 16);
}

constexpr int kThreads = 128;

// A vector (a head's query or key of one map, or a value) is taken by `lanes` neighbouring lanes (a power of two) of 8
// channels each; a thread goes over kRun consecutive rows of the step, its channels' taps read once. A run inside one
// request, behind its first K - 1 rows, has all its rows asked for at once; others slide a window of K registers a channel. Blocks y < qk_blocks take query and key vectors, the rest
// value vectors (which may be of another size).
template <typename T, int K, int kRun>
__global__ void __launch_bounds__(kThreads) conv_qkv_kernel(const ConvArgs a, int qk_blocks, int qk_lanes, int v_lanes) {
  const bool is_v = (int)blockIdx.y >= qk_blocks;
  const int lanes = is_v ? v_lanes : qk_lanes;
  const int per_block = kThreads / lanes;
  const int vec = (is_v ? (int)blockIdx.y - qk_blocks : (int)blockIdx.y) * per_block + (int)threadIdx.x / lanes;
  const int sub = threadIdx.x % lanes;
  const int nq = a.heads * a.maps, nk = a.kv_heads * a.maps;
  const int size = is_v ? a.vdim : a.dim;
  const bool is_q = !is_v && vec < nq;
  const bool exists = vec < (is_v ? a.kv_heads : nq + nk) && (is_q || a.write_kv);
  const bool owns = exists && sub * 8 < size;
  const int c0 = (is_v ? (nq + nk) * a.dim : 0) + vec * size + sub * 8;        // first channel
  const int channels = (nq + nk) * a.dim + a.kv_heads * a.vdim;
  const T* proj = reinterpret_cast<const T*>(a.proj);
  float w[8 * K], nw[8];
#pragma unroll
  for (int i = 0; i < 8 * K; ++i) w[i] = 1.f;                                  // [tap][channel]
  if (owns && a.taps) {
#pragma unroll
    for (int j = 0; j < K; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float4 f = *reinterpret_cast<const float4*>(a.taps + (size_t)j * channels + c0 + 4 * i);
        w[8 * j + 4 * i] = f.x; w[8 * j + 4 * i + 1] = f.y; w[8 * j + 4 * i + 2] = f.z; w[8 * j + 4 * i + 3] = f.w;
      }
  }
  const float* norm_w = is_v ? nullptr : (is_q ? a.q_w : a.k_w);
#pragma unroll
  for (int e = 0; e < 8; ++e) nw[e] = owns && norm_w ? norm_w[sub * 8 + e] : 1.f;
  const int map = is_v ? 0 : (is_q ? vec : vec - nq) % a.maps;
  const int own_at = map * a.dim;                                              // (values: 0)
  // one row's vector: norm, place in its row of q or of the cache
  auto finish = [&](float (&y)[8], float ss, int t, int s, int pos) {
    if (!is_v && a.norm) {                                                     // the same for the whole block
      for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float inv = rsqrtf(ss / (float)size + a.eps);
#pragma unroll
      for (int e = 0; e < 8; ++e) y[e] *= inv * nw[e];
    }
    if (!exists) return;
    T* row;
    if (is_q) {
      row = reinterpret_cast<T*>(a.q_out) + ((size_t)t * nq + vec) * a.hd;
    } else {
      const int page = a.block_table[(size_t)s * a.table_stride + pos / a.page_size];
      if (page < 0) return;                                                    // the host reserves pages before the step
      const int kvh = is_v ? vec : (vec - nq) / a.maps;
      row = reinterpret_cast<T*>(is_v ? a.v_pages : a.k_pages) +
            (((size_t)page * a.kv_heads + kvh) * a.page_size + pos % a.page_size) * a.hd;
    }
    if (owns) store8(row + own_at + sub * 8, y);
    const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (is_q && owns)
      for (int m = 0; m < a.maps; ++m)
        if (m != map) store8(row + m * a.dim + sub * 8, zero);
    if (is_q || map == 0)                                                      // padding behind the maps (or the value)
      for (int d = (is_v ? a.vdim : a.maps * a.dim) + sub * 8; d < a.hd; d += lanes * 8) store8(row + d, zero);
  };
  const int t0 = blockIdx.x * kRun;
  if constexpr (kRun > 1) {
    const int s = a.seq_of_token[t0];
    if (t0 + kRun <= a.n_tokens && t0 - a.cu_seqlens[s] >= K - 1 && t0 + kRun <= a.cu_seqlens[s + 1]) {
      Raw8<T> rows[kRun + K - 1];
      if (owns) {
#pragma unroll
        for (int i = 0; i < kRun + K - 1; ++i) rows[i] = raw8(proj + (size_t)(t0 - (K - 1) + i) * a.ld + c0);
      }
      const int pos0 = a.positions[t0];
#pragma unroll
      for (int i = 0; i < kRun; ++i) {
        float y[8];
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          float acc = 0.f;
          if (owns) {
#pragma unroll
            for (int j = 0; j < K; ++j) acc = fmaf(w[8 * j + e], element(rows[i + j], e), acc);
          }
          y[e] = acc;
          ss += acc * acc;
        }
        finish(y, ss, t0 + i, s, pos0 + i);
      }
      return;
    }
  }
  float x[K][8];
  int prev_seq = -1;
#pragma unroll 1
  for (int i = 0; i < kRun; ++i) {
    const int t = t0 + i;
    if (t >= a.n_tokens) break;                                                // the same for the whole block
    const int s = a.seq_of_token[t];
    if (owns) {
      if (s == prev_seq) {
#pragma unroll
        for (int j = 0; j + 1 < K; ++j)
#pragma unroll
          for (int e = 0; e < 8; ++e) x[j][e] = x[j + 1][e];
        hb::load8(proj + (size_t)t * a.ld + c0, x[K - 1]);
      } else {
        const int start = a.cu_seqlens[s], local = t - start;
        const float* tail = a.state + (K > 1 ? (size_t)a.slots[s] * a.state_stride + a.conv_off : 0);
#pragma unroll
        for (int j = 0; j < K; ++j) {
          const int rel = local - (K - 1) + j;
          if (rel >= 0) hb::load8(proj + (size_t)(start + rel) * a.ld + c0, x[j]);
          else hb::load8(tail + (size_t)(K - 1 + rel) * channels + c0, x[j]);
        }
      }
    }
    prev_seq = s;
    float y[8];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float acc = 0.f;
      if (owns) {
#pragma unroll
        for (int j = 0; j < K; ++j) acc = fmaf(w[8 * j + e], x[j][e], acc);
      }
      y[e] = acc;
      ss += acc * acc;
    }
    finish(y, ss, t, s, a.positions[t]);
    // the request's only token of the step: its inputs move up a row in the state, which this thread alone reads and
    // writes at these channels
    if (K > 1 && a.fuse_tail && owns) {
      float* tail = a.state + (size_t)a.slots[s] * a.state_stride + a.conv_off;
#pragma unroll
      for (int j = 1; j < K; ++j) store8(tail + (size_t)(j - 1) * channels + c0, x[j]);
    }
  }
}

// Any sizes, any number of taps, rotation: a block is one token, a warp takes a vector at a time through a row of
// shared memory. (The state is moved by a launch of its own.)
template <typename T>
__global__ void conv_qkv_general_kernel(const ConvArgs a) {
  extern __shared__ float smem_c[];            // [rot_pairs] cos, [rot_pairs] sin, [warps][max(dim, vdim)]
  float* cs = smem_c;
  float* sn = cs + a.rot_pairs;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  float* row = sn + a.rot_pairs + warp * max(a.dim, a.vdim);
  const int t = blockIdx.x;
  const int s = a.seq_of_token[t], pos = a.positions[t];
  const int start = a.cu_seqlens[s], local = t - start;
  for (int j = threadIdx.x; j < a.rot_pairs; j += blockDim.x) {
    float s_, c_;
    sincosf((float)pos * a.inv_freq[j], &s_, &c_);
    cs[j] = c_ * a.rot_mul;
    sn[j] = s_ * a.rot_mul;
  }
  __syncthreads();
  const int nq = a.heads * a.maps, nk = a.kv_heads * a.maps, rot = 2 * a.rot_pairs;
  const int channels = (nq + nk) * a.dim + a.kv_heads * a.vdim;
  const T* proj = reinterpret_cast<const T*>(a.proj);
  const float* tail = a.K > 1 ? a.state + (size_t)a.slots[s] * a.state_stride + a.conv_off : nullptr;
  for (int vec = warp; vec < nq + nk + a.kv_heads; vec += nwarps) {
    const bool is_v = vec >= nq + nk, is_q = vec < nq;
    if (!is_q && !a.write_kv) break;
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(a.q_out) + ((size_t)t * nq + vec) * a.hd;
    } else {
      const int page = a.block_table[(size_t)s * a.table_stride + pos / a.page_size];
      if (page < 0) continue;
      const int kvh = is_v ? vec - nq - nk : (vec - nq) / a.maps;
      dst = reinterpret_cast<T*>(is_v ? a.v_pages : a.k_pages) +
            (((size_t)page * a.kv_heads + kvh) * a.page_size + pos % a.page_size) * a.hd;
    }
    const int size = is_v ? a.vdim : a.dim;
    const int c0 = is_v ? (nq + nk) * a.dim + (vec - nq - nk) * a.vdim : vec * a.dim;
    float ss = 0.f;
    for (int d = lane; d < size; d += 32) {
      float acc = 0.f;
      if (a.taps) {
        for (int j = 0; j < a.K; ++j) {
          const int rel = local - (a.K - 1) + j;
          const float u = rel >= 0 ? hb::to_f32(proj[(size_t)(start + rel) * a.ld + c0 + d])
                                   : tail[(size_t)(a.K - 1 + rel) * channels + c0 + d];
          acc = fmaf(a.taps[(size_t)j * channels + c0 + d], u, acc);
        }
      } else {
        acc = hb::to_f32(proj[(size_t)t * a.ld + c0 + d]);
      }
      row[d] = acc;
      ss += acc * acc;
    }
    ss = hb::warp_sum(ss);
    __syncwarp();
    const float* w = is_v ? nullptr : (is_q ? a.q_w : a.k_w);
    const float inv = !is_v && a.norm ? rsqrtf(ss / (float)size + a.eps) : 1.f;
    for (int d = lane; d < size; d += 32) row[d] *= inv * (w ? w[d] : 1.f);
    __syncwarp();
    const int map = is_v ? 0 : (is_q ? vec : vec - nq) % a.maps;
    for (int d = lane; d < size; d += 32) {
      float y = row[d];
      if (!is_v && d < rot) {
        if (a.interleaved) {
          const int j = d >> 1;
          y = (d & 1) ? row[d] * cs[j] + row[d - 1] * sn[j] : row[d] * cs[j] - row[d + 1] * sn[j];
        } else {
          y = d < a.rot_pairs ? row[d] * cs[d] - row[d + a.rot_pairs] * sn[d]
                              : row[d] * cs[d - a.rot_pairs] + row[d - a.rot_pairs] * sn[d - a.rot_pairs];
        }
      }
      dst[map * a.dim + d] = hb::from_f32<T>(y);
    }
    if (is_q)
      for (int m = 0; m < a.maps; ++m)
        if (m != map)
          for (int d = lane; d < size; d += 32) dst[m * a.dim + d] = hb::from_f32<T>(0.f);
    if (is_q || map == 0)
      for (int d = (is_v ? a.vdim : a.maps * a.dim) + lane; d < a.hd; d += 32) dst[d] = hb::from_f32<T>(0.f);
    __syncwarp();
  }
}

template <typename T, int kRun>
void launch_run(const ConvArgs& a, dim3 grid, int qk_blocks, int qk_lanes, int v_lanes, cudaStream_t stream) {
  switch (a.K) {
    case 1: conv_qkv_kernel<T, 1, kRun><<<grid, kThreads, 0, stream>>>(a, qk_blocks, qk_lanes, v_lanes); break;
    case 2: conv_qkv_kernel<T, 2, kRun><<<grid, kThreads, 0, stream>>>(a, qk_blocks, qk_lanes, v_lanes); break;
    case 3: conv_qkv_kernel<T, 3, kRun><<<grid, kThreads, 0, stream>>>(a, qk_blocks, qk_lanes, v_lanes); break;
    default: conv_qkv_kernel<T, 4, kRun><<<grid, kThreads, 0, stream>>>(a, qk_blocks, qk_lanes, v_lanes); break;
  }
}

int lanes_for(int size) {
  int lanes = 1;
  while (lanes * 8 < size) lanes *= 2;
  return lanes;
}

template <typename T>
int launch_conv(const ConvArgs& a, bool fast, cudaStream_t stream) {
  if (!fast) {
    const int vectors = (a.heads + a.kv_heads) * a.maps + a.kv_heads;
    const int warps = vectors < 8 ? vectors : 8;
    const size_t smem = (size_t)(2 * a.rot_pairs + warps * (a.dim > a.vdim ? a.dim : a.vdim)) * sizeof(float);
    if (smem > 48 * 1024) return HB_ERR_UNSUPPORTED;
    conv_qkv_general_kernel<T><<<a.n_tokens, warps * 32, smem, stream>>>(a);
    HB_LAUNCH_CHECK();
    return HB_OK;
  }
  const int qk_lanes = lanes_for(a.dim), v_lanes = lanes_for(a.vdim);
  const int qk = (a.heads + a.kv_heads) * a.maps;
  const int qk_blocks = (qk * qk_lanes + kThreads - 1) / kThreads;
  const int v_blocks = a.write_kv ? (a.kv_heads * v_lanes + kThreads - 1) / kThreads : 0;
  if (qk_blocks + v_blocks > 65535) return HB_ERR_UNSUPPORTED;
  // many rows: eight a thread (a row is then loaded once, not K times); few: one, so that the step spreads over the GPU
  if (!a.fuse_tail && (long long)a.n_tokens * (qk_blocks + v_blocks) >= 8 * 148 * 2)
    launch_run<T, 8>(a, dim3((a.n_tokens + 7) / 8, qk_blocks + v_blocks), qk_blocks, qk_lanes, v_lanes, stream);
  else
    launch_run<T, 1>(a, dim3(a.n_tokens, qk_blocks + v_blocks), qk_blocks, qk_lanes, v_lanes, stream);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

}  // namespace

// `taps` [taps_n][channels] float32 or null (no convolution; taps_n is then 1). `single_tokens`: every request of the
// step brings one token. `moved` (host, one int): set to 1 when the kernel moved the requests' inputs in the state
// itself, 0 when the caller has to (hb_delta_conv_update has the state layout's rule).
extern "C" int hb_conv_qkv(const void* proj, int dtype, long long ld, const float* taps, int taps_n, float* state,
                           long long state_stride, long long conv_off, int norm, float eps, const float* q_w,
                           const float* k_w, const float* inv_freq, int rot_pairs, int interleaved, float rot_mul,
                           const int* positions, const int* seq_of_token, const int* cu_seqlens, const int* slots,
                           const int* block_table, int table_stride, void* q_out, void* k_pages, void* v_pages,
                           int page_size, int write_kv, int single_tokens, int n_tokens, int heads, int kv_heads,
                           int maps, int dim, int vdim, int hd, int* moved, cudaStream_t stream) {
  if (!proj || !positions || !seq_of_token || !cu_seqlens || !q_out || !moved || n_tokens < 0 || heads <= 0 || kv_heads <= 0 ||
      maps < 1 || maps > 2 || dim <= 0 || vdim <= 0 || taps_n < 1 || (!taps && taps_n != 1))
    return HB_ERR_BAD_ARG;
  if (taps_n > 1 && (!state || !slots)) return HB_ERR_BAD_ARG;
  if (write_kv && (!k_pages || !v_pages || !block_table || page_size <= 0 || table_stride <= 0)) return HB_ERR_BAD_ARG;
  if (maps * dim > hd || vdim > hd) return HB_ERR_BAD_ARG;
  if (!inv_freq) rot_pairs = 0;
  if (rot_pairs < 0 || 2 * rot_pairs > dim) return HB_ERR_BAD_ARG;
  *moved = 0;
  if (n_tokens == 0) return HB_OK;
  ConvArgs a{};
  a.proj = proj; a.ld = ld; a.taps = taps; a.state = state; a.state_stride = state_stride; a.conv_off = conv_off;
  a.q_w = q_w; a.k_w = k_w; a.inv_freq = inv_freq; a.rot_pairs = rot_pairs; a.interleaved = interleaved;
  a.rot_mul = rot_mul; a.eps = eps; a.norm = norm; a.write_kv = write_kv; a.K = taps_n;
  a.positions = positions; a.seq_of_token = seq_of_token; a.cu_seqlens = cu_seqlens; a.slots = slots;
  a.block_table = block_table; a.table_stride = table_stride; a.page_size = page_size;
  a.q_out = q_out; a.k_pages = k_pages; a.v_pages = v_pages;
  a.n_tokens = n_tokens; a.heads = heads; a.kv_heads = kv_heads; a.maps = maps; a.dim = dim; a.vdim = vdim; a.hd = hd;
  const bool fast = rot_pairs == 0 && taps_n <= 4 && dim % 8 == 0 && vdim % 8 == 0 && hd % 8 == 0 && dim <= 256 && vdim <= 256 &&
                    ld % 8 == 0 && ((uintptr_t)proj & 15) == 0 && state_stride % 4 == 0 && conv_off % 4 == 0 &&
                    ((uintptr_t)state & 15) == 0 && ((uintptr_t)taps & 15) == 0;
  a.fuse_tail = fast && single_tokens && taps_n > 1 ? 1 : 0;
  *moved = a.fuse_tail;
  if (dtype == HB_DTYPE_F32) return launch_conv<float>(a, fast, stream);
  if (dtype == HB_DTYPE_BF16) return launch_conv<__nv_bfloat16>(a, fast, stream);
  return HB_ERR_BAD_ARG;
}
