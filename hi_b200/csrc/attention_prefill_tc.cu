// Prefill attention on the 5th-generation tensor cores (tcgen05), bfloat16: portions of prompts of
// at least a tile of new tokens against the paged cache. One block = 128 consecutive new tokens
// of one request and one query head:
//   warp 0      one lane issues TMA loads: the Q tile once, then K and V tiles of 64 key positions
//               (one box per page, 128-byte swizzle): K into a ring of three and a tile ahead of V,
//               V into a ring of two (a load takes about as long as a tile's work, so with two
//               stages and K and V in turn the products waited for their K: measured 5.76 -> 5.16 ms
//               for 4,096 new tokens behind 61,440);
//   warp 1      allocates tensor memory; one lane issues S = Q K^T (tcgen05.mma, M 128, N 64) into
//               one of two S buffers and, a tile behind, O += P V (P read from tensor memory, where
//               it lies over its own S; V from shared memory as the MN-major operand), so the next
//               S is computed while the softmax works on this one;
//   warps 2..5  softmax: thread r owns row r (tensor-memory lane r): it reads its S row with
//               tcgen05.ld, masks by absolute position (causal, chunk, sliding window), keeps the
//               running max and sum in float32, rescales its O row in tensor memory when the max
//               moved, and writes P as bfloat16 back into tensor memory (tcgen05.st): the products
//               are bound by what the SM can read from shared memory, and P from there would add a
//               fifth to it.
// Differential attention (two maps per head over the same values, maps == 2): one block = 64 new tokens of one request
// and BOTH maps of a head. Row r of the tile is token r % 64 of map r / 64, so the two maps share every key and value
// tile, and the epilogue subtracts them, norms the head's row and gates it before it leaves (see Pair).
// A window that keeps the first tokens of a request (keep > 0) walks the tiles of the kept tokens first.
// Every mbarrier wait is bounded; on a time-out a code goes to `status` and the block leaves
// through the common exit, where tensor memory is freed.
#include <cuda.h>
#include <cuda_bf16.h>
#include <stdint.h>

#include "api.h"
#include "common.cuh"
#include "tc.cuh"

namespace {

constexpr int BQ = 128;          // query rows per block (UMMA M)
constexpr int KST = 3;           // K tiles in flight
constexpr int BKEYS = 64;        // key positions per tile (two blocks per SM then fit: one does MMAs while the other's softmax runs)
constexpr int THREADS = 192;

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// What the epilogue does with the two maps a1, a2 of a head (float32, normalised by their softmax):
//   o = a1 - lambda a2;  o <- o rsqrt(mean over vdim of o^2 + eps) mul;  out = o * sigmoid(gate)   (gate null: no gate)
// `out` is [rows, nh / 2, vdim]; gate row t starts at gate + t * gate_stride and is laid out as a row of `out`.
struct Pair {
  float lambda, eps, mul;
  int vdim, vec;                 // vec: vdim, the rows of `out` and of the gate allow 16-byte accesses
  const __nv_bfloat16* gate;
  long long gate_stride;
};

struct Args {
  const int* block_table;
  const int* cu_seqlens;
  const int* positions;
  __nv_bfloat16* out;
  int* status;
  int table_stride, nh, nkv, page_size, chunk, window, skip_single, box_rows;
  float scale_log2;          // softmax scale * log2(e)
  // With key_splits > 1 every (query tile, head) is `key_splits` blocks, each over its share of the
  // key tiles; a block leaves its rows unnormalised in part_acc [row][split][head_dim] with (max,
  // sum) in part_ml [row][split][2] (max in natural-log units), and hb_attention_merge combines them.
  int key_splits;
  float* part_acc;
  float* part_ml;
  int sink;                  // 1: the denominator has one more term, e^0 (a key of score 0 without a value)
  // sink == 2: sigmoid weights. A key weighs sigmoid(score + head_bias[head]) = 1 / (1 + 2^-(raw * scale_log2 +
  // bias * log2 e)); nothing is normalised; every block leaves its plain sums in part_acc (zero-filled by the
  // caller, also with key_splits == 1) and the caller adds the splits.
  const float* head_bias;
  // turn_inside (sigmoid weights, key_splits == 1): the block turns its rows back itself and writes `out`. The
  // values were cached rotated by their own positions: pair m of the row's first 2 * v_pairs dims (interleaved:
  // dims 2m, 2m + 1; else m, m + v_pairs with 2 * v_pairs == head_dim) turns by -position * v_inv_freq[m].
  int turn_inside, v_pairs, v_interleaved;
  const float* v_inv_freq;
  // Scores reshaped before the softmax: softcap > 0: s <- softcap tanh(s / softcap) on the scaled score; slopes [nh]
  // (or null): slopes[head] * (query position - key position) is taken off after the cap. sink_values [nh] (or
  // null): with sink == 1 the extra term's score is the head's own number instead of 0.
  float softcap;
  const float* slopes;
  const float* sink_values;
  // With a distance bias the newest keys score highest: the key tiles are then taken newest first, so that the running
  // maximum is found in the first tiles and O is seldom rescaled (oldest first it would move with nearly every tile).
  int newest_first;
  int keep;                  // a sliding window's kept first tokens
  Pair pair;                 // kPair only
};

template <int HD, bool kPair>
__global__ void __launch_bounds__(THREADS, 2)
attn_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                       const __grid_constant__ CUtensorMap map_v, const Args a) {
  constexpr int DBLK = HD / 64;                 // 64-dim blocks of a row
  constexpr int QBYTES = BQ * HD * 2, KBYTES = BKEYS * HD * 2;
  constexpr int QBLOCK = BQ * 128;              // bytes of one [128 rows x 64 elements] swizzled block of Q
  constexpr int KVBLOCK = BKEYS * 128;          // the same for a K or V tile (rows = key positions)
  constexpr int S_COLS = BKEYS;                 // columns of one S buffer
  // S0, S1 (64 columns each), O (HD columns); an allocation is a power of two. Rows over 128 take the whole
  // tensor memory of the SM, where their shared memory lets one block live anyway.
  constexpr int TMEM_COLS = 2 * S_COLS + HD <= 256 ? 256 : 512;
  static_assert(HD % 64 == 0 && 2 * S_COLS + HD <= 512, "rows of 64-element blocks, S and O within tensor memory");
  // No slack for aligning by hand: two blocks per SM only fit without it. The swizzled tiles need
  // a 1024-byte aligned base, which dynamic shared memory has when the kernel has no static
  // shared memory; if it ever has not, the block reports it and leaves.
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;
  if ((tc::smem_u32(smem) & 1023u) != 0) {
    if (threadIdx.x == 0) atomicExch(a.status, 19);
    return;
  }
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + QBYTES;                  // [KST stages] K tiles
  uint8_t* v_s = k_s + KST * KBYTES;            // [2 stages] V tiles
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + 2 * KBYTES);
  uint64_t* q_full = bars;            // 1
  uint64_t* k_full = bars + 1;        // 3   K and V have rings of their own: a K buffer is free as soon
  uint64_t* k_empty = bars + 4;       // 3   as its S is computed, long before its V is used, and K is
  uint64_t* v_full = bars + 7;        // 2   loaded a tile ahead of V
  uint64_t* v_empty = bars + 9;       // 2
  uint64_t* s_full = bars + 11;       // 2
  uint64_t* s_free = bars + 13;       // 2
  uint64_t* p_ready = bars + 15;      // 1
  uint64_t* pv_done = bars + 16;      // 1
  uint64_t* ex_ready = bars + 17;     // 1   kPair: the maps' halves, then their sums of squares, are in shared memory
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
  constexpr int kst = KST;
  constexpr int TOKENS = kPair ? BQ / 2 : BQ;   // new tokens of a block

  // Blocks start in the order x, y, z: the heads are x and the query tiles y, latest first, so
  // the tiles that read the most keys start first for every head and the short ones fill the end.
  const int heads = kPair ? a.nh / 2 : a.nh;
  const int seq = blockIdx.z, h = blockIdx.x % heads, piece = blockIdx.x / heads;
  const int qt = gridDim.y - 1 - blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq_begin = a.cu_seqlens[seq], seq_end = a.cu_seqlens[seq + 1];
  const int tok0 = seq_begin + qt * TOKENS;
  const int n_valid = min(TOKENS, seq_end - tok0);
  if (n_valid <= 0) return;
  // a row that this block leaves out weighs nothing in the merge
  const bool sigmoid = a.sink == 2;
  auto no_part = [&](int row) {
    if (sigmoid) return;                        // part_acc was zero-filled: the row adds nothing
    float* ml = a.part_ml + (((size_t)(tok0 + row) * a.nh + h) * a.key_splits + piece) * 2;
    ml[0] = -INFINITY;
    ml[1] = 0.f;
  };
  if (a.skip_single && seq_end - seq_begin == 1) {
    if (a.key_splits > 1 && threadIdx.x == 0) no_part(0);
    return;
  }
  const int kvh = (kPair ? 2 * h : h) / (a.nh / a.nkv);
  const int p_first = a.positions[tok0];
  const int p_last = p_first + n_valid - 1;
  auto first_visible = [&](int pos) {
    int lo = 0;
    if (a.chunk > 0) lo = (pos / a.chunk) * a.chunk;
    if (a.window > 0 && pos - a.window + 1 > lo) lo = pos - a.window + 1;
    return lo;
  };
  int tile_begin = first_visible(p_first) / BKEYS;
  // the walk: tiles of kept tokens before the window's first tile, then the window's
  const int kept_tiles = a.keep > 0 ? min((a.keep + BKEYS - 1) / BKEYS, tile_begin) : 0;
  int nt = kept_tiles + p_last / BKEYS - tile_begin + 1;
  if (a.key_splits > 1) {                       // this block's share of the key tiles
    const int share = (nt + a.key_splits - 1) / a.key_splits;
    tile_begin += piece * share;
    nt = min(share, nt - piece * share);
    if (nt <= 0) {
      if ((int)threadIdx.x < n_valid) no_part(threadIdx.x);
      return;
    }
  }
  auto tile_key0 = [&](int j) {                 // first key position of the j-th tile of this block
    const int w = a.newest_first ? nt - 1 - j : j;
    return (w < kept_tiles ? w : tile_begin + w - kept_tiles) * BKEYS;
  };

  if (threadIdx.x == 0) {
    tc::mbar_init(q_full, 1);
    for (int i = 0; i < KST; ++i) { tc::mbar_init(&k_full[i], 1); tc::mbar_init(&k_empty[i], 1); }
    for (int i = 0; i < 2; ++i) {
      tc::mbar_init(&v_full[i], 1); tc::mbar_init(&v_empty[i], 1);
      tc::mbar_init(&s_full[i], 1); tc::mbar_init(&s_free[i], 4);
    }
    tc::mbar_init(p_ready, 4);
    tc::mbar_init(pv_done, 1);
    tc::mbar_init(ex_ready, 4);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    tc::alloc(tmem_slot, TMEM_COLS);
  }
  tc::fence_before();
  __syncthreads();
  tc::fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t tmem_o = tmem + 2 * S_COLS;

  if (warp == 0) {
    if (lane == 0) {                            // ---- TMA producer
      const int* table = a.block_table + (size_t)seq * a.table_stride;
      tc::mbar_expect_tx(q_full, QBYTES);
      if (kPair) {                              // the box is 64 rows: map 1 above map 2 in every 64-element block
        for (int c = 0; c < DBLK; ++c)
          for (int mp = 0; mp < 2; ++mp)
            tc::tma_load_2d(q_s + c * QBLOCK + mp * (QBLOCK / 2), &map_q, (2 * h + mp) * HD + c * 64, tok0, q_full);
      } else {
        for (int c = 0; c < DBLK; ++c) tc::tma_load_2d(q_s + c * QBLOCK, &map_q, h * HD + c * 64, tok0, q_full);
      }
      const int boxes = BKEYS / a.box_rows;
      bool ok = true;
      // one tile of K or V: a box per page
      auto load = [&](int j, uint8_t* dst, const CUtensorMap* map, uint64_t* full) {
        tc::mbar_expect_tx(full, KBYTES);
        for (int b = 0; b < boxes; ++b) {
          const int key0 = tile_key0(j) + b * a.box_rows;
          const int page = key0 <= p_last ? table[key0 / a.page_size] : -1;
          // keys past the portion's last position (or without a page) are masked: any row will do
          const int row = page >= 0 ? (page * a.nkv + kvh) * a.page_size + key0 % a.page_size : 0;
          for (int c = 0; c < DBLK; ++c) tc::tma_load_2d(dst + c * KVBLOCK + b * a.box_rows * 128, map, c * 64, row, full);
        }
      };
      auto load_k = [&](int j) {
        const int s = j % kst, use = j / kst;
        if (use >= 1 && !tc::mbar_wait(&k_empty[s], (use - 1) & 1)) { atomicExch(a.status, 11); ok = false; return; }
        load(j, k_s + s * KBYTES, &map_k, &k_full[s]);
      };
      auto load_v = [&](int j) {
        const int s = j & 1;
        if (j >= 2 && !tc::mbar_wait(&v_empty[s], ((j >> 1) - 1) & 1)) { atomicExch(a.status, 20); ok = false; return; }
        load(j, v_s + s * KBYTES, &map_v, &v_full[s]);
      };
      load_k(0);
      for (int j = 0; j < nt && ok; ++j) {          // K runs a tile ahead of V
        if (j + 1 < nt) load_k(j + 1);
        if (ok) load_v(j);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {                            // ---- MMA issuer: S_j = Q K_j^T, then O += P_{j-1} V_{j-1}
      constexpr uint32_t idesc_qk = tc::idesc_bf16(BQ, BKEYS, false);
      constexpr uint32_t idesc_pv = tc::idesc_bf16(BQ, HD, true);
      bool ok = tc::mbar_wait(q_full, 0);
      if (!ok) atomicExch(a.status, 12);
      tc::fence_after();
      const uint32_t q_addr = tc::smem_u32(q_s);
      for (int j = 0; j <= nt && ok; ++j) {
        if (j < nt) {
          const int s = j & 1;
          const int ks = j % kst;
          if (!tc::mbar_wait(&k_full[ks], (j / kst) & 1)) { atomicExch(a.status, 13); ok = false; break; }
          if (j >= 2 && !tc::mbar_wait(&s_free[s], ((j >> 1) - 1) & 1)) { atomicExch(a.status, 14); ok = false; break; }
          // S_j goes where P_{j-2} lies: the product that reads that P must be through (it is the last one
          // committed to this barrier so far, so the parity is its own)
          if (j >= 2 && !tc::mbar_wait(pv_done, (j - 2) & 1)) { atomicExch(a.status, 24); ok = false; break; }
          tc::fence_after();
          const uint32_t k_addr = tc::smem_u32(k_s + ks * KBYTES);
#pragma unroll
          for (int k = 0; k < HD / 16; ++k) {
            tc::mma(tmem + s * S_COLS, tc::desc_kmajor(q_addr + (k / 4) * QBLOCK + (k % 4) * 32),
                   tc::desc_kmajor(k_addr + (k / 4) * KVBLOCK + (k % 4) * 32), idesc_qk, k != 0);
          }
          tc::commit(&s_full[s]);
          tc::commit(&k_empty[ks]);             // the K buffer is free once these MMAs have read it
        }
        if (j >= 1) {
          const int i = j - 1, s = i & 1;
          if (!tc::mbar_wait(&v_full[s], (i >> 1) & 1)) { atomicExch(a.status, 21); ok = false; break; }
          if (!tc::mbar_wait(p_ready, i & 1)) { atomicExch(a.status, 15); ok = false; break; }
          tc::fence_after();
          const uint32_t v_addr = tc::smem_u32(v_s + s * KBYTES);
          const uint32_t p_tmem = tmem + s * S_COLS;     // P_i lies over the first half of S_i's columns
#pragma unroll
          for (int k = 0; k < BKEYS / 16; ++k) {
            tc::mma_a_tmem(tmem_o, p_tmem + k * 8, tc::desc_mnmajor(v_addr + k * 2048, KVBLOCK), idesc_pv, (i | k) != 0);
          }
          tc::commit(&v_empty[s]);
          tc::commit(pv_done);
        }
      }
    }
  } else {                                      // ---- softmax: thread = row = tensor-memory lane
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const uint32_t lane_addr = (uint32_t)(quarter * 32) << 16;
    const int row = kPair ? r % TOKENS : r;     // this row's token within the block
    const int warp_row = kPair ? (quarter & 1) * 32 : quarter * 32;
    const bool row_ok = row < n_valid;
    const int pos = p_first + row;
    const int lo = first_visible(pos);
    float m = -INFINITY, l = 0.f;
    const float bias_log2 = (sigmoid && a.head_bias) ? a.head_bias[h] * 1.4426950408889634f : 0.f;
    // reshaped scores are brought to units of log 2 first and the code below then takes them with a scale of one
    const bool reshaped = a.softcap > 0.f || a.slopes != nullptr;
    const float scale_l2 = reshaped ? 1.f : a.scale_log2;
    const float slope_l2 = a.slopes ? a.slopes[h] * 1.4426950408889634f : 0.f;
    const float cap_l2 = a.softcap * 1.4426950408889634f;
    const float twice_over_cap = a.softcap > 0.f ? 2.f * a.scale_log2 / a.softcap : 0.f;
    bool ok = true;
    for (int j = 0; j < nt && ok; ++j) {
      const int sb = j & 1;
      if (!__all_sync(0xffffffffu, tc::mbar_wait(&s_full[sb], (j >> 1) & 1))) {
        if (lane == 0) atomicExch(a.status, 16);
        ok = false;
        break;
      }
      tc::fence_after();
      const int key_base = tile_key0(j);
      // a tile every row of this warp sees whole needs no masks (most tiles of a long prompt)
      const int warp_first_pos = p_first + warp_row;
      const bool interior = (warp_row + 31 < n_valid) && (key_base + BKEYS - 1 <= warp_first_pos) &&
                            (key_base >= first_visible(warp_first_pos + 31) || key_base + BKEYS <= a.keep);
      float sv[BKEYS];
      float mx = m;
      {
        // the whole S row: both loads in flight, one wait
        uint32_t raw0[32], raw1[32];
        tc::ld32_nowait(tmem + lane_addr + sb * S_COLS, raw0);
        tc::ld32_nowait(tmem + lane_addr + sb * S_COLS + 32, raw1);
        tc::wait_ld();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          sv[i] = __uint_as_float(raw0[i]);
          sv[32 + i] = __uint_as_float(raw1[i]);
        }
      }
      if (reshaped) {
        // score' = cap tanh(score / cap) - slope * (pos - key), in units of log 2, with tanh(y) = 1 - 2 / (1 + e^(2 y)):
        // one ex2, one reciprocal and three multiply-adds per score; the branches are outside the loops
        const float base = cap_l2 - slope_l2 * (float)(pos - key_base);      // cap_l2 is 0 without a cap
        if (a.softcap > 0.f) {
          const float minus_two_cap = -2.f * cap_l2;
#pragma unroll
          for (int i = 0; i < BKEYS; ++i) {
            float r;
            asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + fast_exp2(sv[i] * twice_over_cap)));
            sv[i] = fmaf(r, minus_two_cap, fmaf(slope_l2, (float)i, base));
          }
        } else {
#pragma unroll
          for (int i = 0; i < BKEYS; ++i) sv[i] = fmaf(sv[i], a.scale_log2, fmaf(slope_l2, (float)i, base));
        }
      }
      if (interior && sigmoid) {
        // nothing to mask and no maximum to follow
      } else if (interior) {
        float top = -INFINITY;
#pragma unroll
        for (int i = 0; i < BKEYS; ++i) top = fmaxf(top, sv[i]);
        mx = fmaxf(mx, top * scale_l2);     // the scale is positive
      } else {
#pragma unroll
        for (int i = 0; i < BKEYS; ++i) {
          const int key = key_base + i;
          // masked scores become -inf BEFORE scaling, so the same exponential code serves both paths
          const float s = (row_ok && key <= pos && (key >= lo || key < a.keep)) ? sv[i] : -INFINITY;
          sv[i] = s;
          mx = fmaxf(mx, s * scale_l2);
        }
      }
      // the S buffer may be overwritten by the MMA two tiles on
      tc::fence_before();
      __syncwarp();
      if (lane == 0) tc::mbar_arrive(&s_free[sb]);
      // The exponentials are taken against `m`, which follows the true running max lazily: it
      // moves (and O and l are rescaled) only when some row of the warp has grown by more than
      // 2^8, so P stays below 256 and most tiles skip the pass over O. The result is the same
      // sum, scaled by a common factor that the final division removes.
      const bool move = !sigmoid && __any_sync(0xffffffffu, mx > m + 8.f || m == -INFINITY);
      float corr = 1.f;
      if (move) {
        corr = (m == -INFINITY) ? 0.f : fast_exp2(m - mx);
        m = mx;
      }
      // p = 2^(raw * scale - m): one fused multiply-add and one ex2 per score; a masked score is
      // -inf and gives 0 (m is finite here unless the whole row is still masked)
      float sum = 0.f;
      if (sigmoid) {
        // p = 1 / (1 + 2^-(raw * scale_log2 + bias_log2)); a masked score is -inf: 2^inf = inf and p = 0
#pragma unroll
        for (int i = 0; i < BKEYS; ++i)
          sv[i] = __fdividef(1.f, 1.f + fast_exp2(-fmaf(sv[i], a.scale_log2, bias_log2)));
      } else if (m == -INFINITY) {
#pragma unroll
        for (int i = 0; i < BKEYS; ++i) sv[i] = 0.f;
      } else {
        // two scores an instruction where the hardware has it (fma and add on pairs of floats);
        // the sum runs in four chains
        const float2 scale2 = make_float2(scale_l2, scale_l2), neg_m2 = make_float2(-m, -m);
        float2 part[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
        for (int i = 0; i < BKEYS; i += 4) {
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const float2 x = __ffma2_rn(make_float2(sv[i + 2 * c], sv[i + 2 * c + 1]), scale2, neg_m2);
            const float2 p = make_float2(fast_exp2(x.x), fast_exp2(x.y));
            sv[i + 2 * c] = p.x;
            sv[i + 2 * c + 1] = p.y;
            part[c] = __fadd2_rn(part[c], p);
          }
        }
        const float2 both = __fadd2_rn(part[0], part[1]);
        sum = both.x + both.y;
      }
      l = l * corr + sum;
      if (j > 0) {
        // The previous P V product must have finished: O is stable. The wait also keeps the warps
        // and the MMA issuer within a tile of one another: that product started only after every
        // warp had handed over its P of the tile before and the issuer had seen it, so the one
        // barrier that counts the hand-overs tile after tile never runs a phase ahead of anyone.
        if (!__all_sync(0xffffffffu, tc::mbar_wait(pv_done, (j - 1) & 1))) {
          if (lane == 0) atomicExch(a.status, 17);
          ok = false;
          break;
        }
        tc::fence_after();
        if (move) {
#pragma unroll 1
          for (int c = 0; c < HD; c += 32) {
            float o[32];
            tc::ld32(tmem_o + lane_addr + c, o);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] *= corr;
            tc::st32(tmem_o + lane_addr + c, o);
          }
        }
      }
      // P row r as bfloat16 goes back into tensor memory, over the first 32 columns of the S row it
      // was made from (two keys a column): the P V product takes it from there as its A operand,
      // so P costs no shared-memory traffic. The product that read the P two tiles ago from these
      // columns ran before the Q K^T that refilled them (one thread issues them, in that order).
      {
        uint32_t packed[BKEYS / 2];
#pragma unroll
        for (int i = 0; i < BKEYS / 2; ++i) {
          __nv_bfloat162 hh = __floats2bfloat162_rn(sv[2 * i], sv[2 * i + 1]);
          packed[i] = *reinterpret_cast<uint32_t*>(&hh);
        }
        tc::st32_nowait(tmem + lane_addr + sb * S_COLS, packed);
        tc::wait_st();
      }
      const bool ragged = key_base / BKEYS == p_last / BKEYS && (p_last + 1) % BKEYS != 0;
      // pages smaller than a tile: the window's first tile and the last tile of kept tokens may hold pages that were given back
      const int walked = a.newest_first ? nt - 1 - j : j;
      const bool holes = a.page_size < BKEYS && (walked == kept_tiles || walked + 1 == kept_tiles);
      if (ragged || holes) {
        // Value rows of positions past the portion's end hold whatever the page held before, and those of pages that
        // were given back are any page's (another request's numbers, possibly not finite): P is zero there, but
        // 0 x NaN is NaN. Once the V tile has landed, the threads of those rows zero them.
        if (!__all_sync(0xffffffffu, tc::mbar_wait(&v_full[sb], (j >> 1) & 1))) {
          if (lane == 0) atomicExch(a.status, 22);
          ok = false;
          break;
        }
        if (r < BKEYS && (key_base + r > p_last ||
                          (holes && a.block_table[(size_t)seq * a.table_stride + (key_base + r) / a.page_size] < 0))) {
          uint8_t* vrow = v_s + sb * KBYTES + (r / 8) * 1024 + (r % 8) * 128;
#pragma unroll
          for (int blk = 0; blk < DBLK; ++blk)
#pragma unroll
            for (int q = 0; q < 8; ++q) *reinterpret_cast<uint4*>(vrow + blk * KVBLOCK + q * 16) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");   // generic writes -> visible to the MMA
      }
      tc::fence_before();
      __syncwarp();
      if (lane == 0) tc::mbar_arrive(p_ready);
    }
    if (ok) {
      if (!__all_sync(0xffffffffu, tc::mbar_wait(pv_done, (nt - 1) & 1))) {
        if (lane == 0) atomicExch(a.status, 18);
      } else {
        tc::fence_after();
        if constexpr (kPair) {
          // The maps trade halves through shared memory (the K tiles are through): row (token, map 1) finishes the
          // first half of the head's values, row (token, map 2) the second; their sums of squares meet there too.
          constexpr int HALF = HD / 2, EXS = HALF + 1;
          float* ex = reinterpret_cast<float*>(k_s);           // [2 maps][64 tokens][EXS]
          float* ex_ss = ex + 2 * TOKENS * EXS;                // [2][64]
          static_assert((2 * TOKENS * EXS + 2 * TOKENS) * 4 <= KST * KBYTES, "the exchange fits the K tiles");
          const int mp = r / TOKENS;
          const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll 1
          for (int c = 0; c < HALF; c += 32) {
            float o[32];
            tc::ld32(tmem_o + lane_addr + (1 - mp) * HALF + c, o);
#pragma unroll
            for (int i = 0; i < 32; ++i) ex[(mp * TOKENS + row) * EXS + c + i] = o[i] * inv;
          }
          __syncwarp();
          if (lane == 0) tc::mbar_arrive(ex_ready);
          bool met = __all_sync(0xffffffffu, tc::mbar_wait(ex_ready, 0));
          float v[HALF];
          float ss = 0.f;
          if (met) {
#pragma unroll
            for (int c = 0; c < HALF; c += 32) {
              float o[32];
              tc::ld32(tmem_o + lane_addr + mp * HALF + c, o);
#pragma unroll
              for (int i = 0; i < 32; ++i) {
                const float mine = o[i] * inv, other = ex[((1 - mp) * TOKENS + row) * EXS + c + i];
                const float d = mp == 0 ? mine - a.pair.lambda * other : other - a.pair.lambda * mine;
                v[c + i] = d;
                ss += d * d;
              }
            }
            ex_ss[mp * TOKENS + row] = ss;
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(ex_ready);
            met = __all_sync(0xffffffffu, tc::mbar_wait(ex_ready, 1));
          }
          if (!met) {
            if (lane == 0) atomicExch(a.status, 23);
          } else if (row_ok) {
            const float total = ex_ss[row] + ex_ss[TOKENS + row];
            const float mul = rsqrtf(total / (float)a.pair.vdim + a.pair.eps) * a.pair.mul;
            __nv_bfloat16* dst = a.out + ((size_t)(tok0 + row) * heads + h) * a.pair.vdim;
            const __nv_bfloat16* gate =
                a.pair.gate ? a.pair.gate + (size_t)(tok0 + row) * a.pair.gate_stride + (size_t)h * a.pair.vdim : nullptr;
#pragma unroll
            for (int c = 0; c < HALF; c += 8) {
              const int d0 = mp * HALF + c;
              if (d0 >= a.pair.vdim) continue;
              float g[8];
              if (a.pair.vec) {                 // vdim is a multiple of 8: the run is whole
                if (gate) hb::load8(gate + d0, g);
              } else if (gate) {
#pragma unroll
                for (int e = 0; e < 8; ++e) g[e] = d0 + e < a.pair.vdim ? __bfloat162float(gate[d0 + e]) : 0.f;
              }
#pragma unroll
              for (int e = 0; e < 8; ++e) {
                v[c + e] *= mul;
                if (gate) v[c + e] *= __fdividef(1.f, 1.f + __expf(-g[e]));
              }
              if (a.pair.vec) {
                uint4 pack;
                uint32_t* w = reinterpret_cast<uint32_t*>(&pack);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  __nv_bfloat162 hh = __floats2bfloat162_rn(v[c + 2 * e], v[c + 2 * e + 1]);
                  w[e] = *reinterpret_cast<uint32_t*>(&hh);
                }
                *reinterpret_cast<uint4*>(dst + d0) = pack;
              } else {
#pragma unroll
                for (int e = 0; e < 8; ++e)
                  if (d0 + e < a.pair.vdim) dst[d0 + e] = __float2bfloat16_rn(v[c + e]);
              }
            }
          }
        } else if (sigmoid && a.turn_inside) {
          // the plain sum is the result: turned back by the row's position in float32, rounded once
          __nv_bfloat16* dst = a.out + ((size_t)(tok0 + r) * a.nh + h) * HD;
          const float fpos = (float)pos;
          auto store32 = [&](const float* o, int c) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              uint4 pack;
              uint32_t* w = reinterpret_cast<uint32_t*>(&pack);
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                __nv_bfloat162 hh = __floats2bfloat162_rn(o[i + 2 * e], o[i + 2 * e + 1]);
                w[e] = *reinterpret_cast<uint32_t*>(&hh);
              }
              *reinterpret_cast<uint4*>(dst + c + i) = pack;
            }
          };
          if (a.v_interleaved || a.v_pairs == 0) {
#pragma unroll 1
            for (int c = 0; c < HD; c += 32) {
              float o[32];
              tc::ld32(tmem_o + lane_addr + c, o);
              if (row_ok) {
#pragma unroll
                for (int e = 0; e < 16; ++e) {
                  const int mth = c / 2 + e;
                  if (mth < a.v_pairs) {
                    float sn, cs;
                    sincosf(fpos * a.v_inv_freq[mth], &sn, &cs);
                    const float u = o[2 * e], v = o[2 * e + 1];
                    o[2 * e] = u * cs + v * sn;
                    o[2 * e + 1] = v * cs - u * sn;
                  }
                }
                store32(o, c);
              }
            }
          } else {
#pragma unroll 1
            for (int c = 0; c < HD / 2; c += 32) {
              float lo[32], hi[32];
              tc::ld32(tmem_o + lane_addr + c, lo);
              tc::ld32(tmem_o + lane_addr + HD / 2 + c, hi);
              if (row_ok) {
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                  float sn, cs;
                  sincosf(fpos * a.v_inv_freq[c + i], &sn, &cs);
                  const float u = lo[i], v = hi[i];
                  lo[i] = u * cs + v * sn;
                  hi[i] = v * cs - u * sn;
                }
                store32(lo, c);
                store32(hi, HD / 2 + c);
              }
            }
          }
        } else if (a.key_splits > 1 || sigmoid) {
          // this share of the keys only: the row as it is, with its max and sum, for the merge
          const size_t at = ((size_t)(tok0 + r) * a.nh + h) * a.key_splits + piece;
          if (row_ok && !sigmoid) {
            a.part_ml[at * 2] = m == -INFINITY ? -INFINITY : m * 0.6931471805599453f;
            a.part_ml[at * 2 + 1] = l;
          }
#pragma unroll 1
          for (int c = 0; c < HD; c += 32) {
            float o[32];
            tc::ld32(tmem_o + lane_addr + c, o);
            if (row_ok) {
              float4* dst4 = reinterpret_cast<float4*>(a.part_acc + at * HD + c);
#pragma unroll
              for (int i = 0; i < 8; ++i) dst4[i] = make_float4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]);
            }
          }
        } else {
        if (a.sink && l > 0.f) l += exp2f((a.sink_values ? a.sink_values[h] * 1.4426950408889634f : 0.f) - m);   // m is in units of log 2
        const float inv = l > 0.f ? 1.f / l : 0.f;
        __nv_bfloat16* dst = a.out + ((size_t)(tok0 + r) * a.nh + h) * HD;
#pragma unroll 1
        for (int c = 0; c < HD; c += 32) {
          float o[32];
          tc::ld32(tmem_o + lane_addr + c, o);
          if (row_ok) {
#pragma unroll
            for (int i = 0; i < 32; i += 8) {
              uint4 pack;
              uint32_t* w = reinterpret_cast<uint32_t*>(&pack);
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                __nv_bfloat162 hh = __floats2bfloat162_rn(o[i + 2 * e] * inv, o[i + 2 * e + 1] * inv);
                w[e] = *reinterpret_cast<uint32_t*>(&hh);
              }
              *reinterpret_cast<uint4*>(dst + c + i) = pack;
            }
          }
        }
        }
      }
    }
  }
  tc::fence_before();
  __syncthreads();
  if (warp == 1) {
    tc::fence_after();
    tc::dealloc(tmem, TMEM_COLS);
  }
}

template <int HD, bool kPair = false>
int launch(const void* q, const void* k_pages, const void* v_pages, const Args& a, int n_tokens, long long pool_rows,
           int n_seqs, int max_new, cudaStream_t stream) {
  CUtensorMap mq, mk, mv;
  if (!tc::make_map_bf16(&mq, q, (uint64_t)n_tokens, (uint64_t)a.nh * HD, kPair ? BQ / 2 : BQ) ||
      !tc::make_map_bf16(&mk, k_pages, (uint64_t)pool_rows, HD, a.box_rows) ||
      !tc::make_map_bf16(&mv, v_pages, (uint64_t)pool_rows, HD, a.box_rows))
    return HB_ERR_UNSUPPORTED;
  const size_t smem = (size_t)BQ * HD * 2 + (KST + 2) * (size_t)BKEYS * HD * 2 + 256;
  cudaError_t e = cudaFuncSetAttribute(attn_prefill_tc_kernel<HD, kPair>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const int tokens = kPair ? BQ / 2 : BQ;
  const int q_tiles = (max_new + tokens - 1) / tokens;
  if (q_tiles > 65535 || n_seqs > 65535) return HB_ERR_UNSUPPORTED;
  if ((long long)a.nh * a.key_splits > 0x7fffffffLL) return HB_ERR_UNSUPPORTED;
  dim3 grid((kPair ? a.nh / 2 : a.nh) * a.key_splits, q_tiles, n_seqs);
  attn_prefill_tc_kernel<HD, kPair><<<grid, THREADS, smem, stream>>>(mq, mk, mv, a);
  HB_LAUNCH_CHECK();
  return HB_OK;
}

}  // namespace

// bfloat16, head_dim 64, 128 or 192, page_size a multiple of 16 that divides 64 or is a multiple of it.
// Arguments as hb_attention_prefill, plus the number of rows of `q`, the number of pages of the
// pools, `key_splits` (1, or how many blocks share the key tiles of a query tile and head: the rows
// then go unnormalised to `part_acc` [n_tokens * nh][key_splits][hd] and `part_ml`
// [n_tokens * nh][key_splits][2] for hb_attention_merge, and `out` is not written), and `status` (one int on the device, zero before the call; nonzero afterwards = a wait
// timed out). HB_ERR_UNSUPPORTED for other shapes: the caller uses hb_attention_prefill.
namespace {
int prefill_tc(const void* q, const void* k_pages, const void* v_pages, const int* block_table, int table_stride,
               const int* cu_seqlens, const int* positions, void* out, int n_tokens, int n_pages, int n_seqs, int max_new,
               int nh, int nkv, int hd, int page_size, int chunk, int window, float scale, int skip_single, int sink,
               const float* head_bias, int key_splits, float* part_acc, float* part_ml, int* status, int turn_inside,
               const float* v_inv_freq, int v_pairs, int v_interleaved, float softcap, const float* slopes,
               const float* sink_values, int keep, const Pair* pair, cudaStream_t stream);
}  // namespace

extern "C" int hb_attention_prefill_tc(const void* q, const void* k_pages, const void* v_pages, const int* block_table,
                                       int table_stride, const int* cu_seqlens, const int* positions, void* out,
                                       int n_tokens, int n_pages, int n_seqs, int max_new, int nh, int nkv, int hd,
                                       int page_size, int chunk, int window, float scale, int skip_single,
                                       int sink, const float* head_bias, int key_splits, float* part_acc,
                                       float* part_ml, int* status, cudaStream_t stream) {
  return prefill_tc(q, k_pages, v_pages, block_table, table_stride, cu_seqlens, positions, out, n_tokens, n_pages, n_seqs,
                    max_new, nh, nkv, hd, page_size, chunk, window, scale, skip_single, sink, head_bias, key_splits,
                    part_acc, part_ml, status, 0, nullptr, 0, 0, 0.f, nullptr, nullptr, 0, nullptr, stream);
}

// The same with reshaped scores (see Args): a cap, a distance bias per head, a sink with a score per head.
extern "C" int hb_attention_prefill_tc_reshaped(const void* q, const void* k_pages, const void* v_pages,
                                                const int* block_table, int table_stride, const int* cu_seqlens,
                                                const int* positions, void* out, int n_tokens, int n_pages, int n_seqs,
                                                int max_new, int nh, int nkv, int hd, int page_size, int chunk,
                                                int window, int keep, float scale, int skip_single, int sink, float softcap,
                                                const float* slopes, const float* sink_values, int key_splits,
                                                float* part_acc, float* part_ml, int* status, cudaStream_t stream) {
  return prefill_tc(q, k_pages, v_pages, block_table, table_stride, cu_seqlens, positions, out, n_tokens, n_pages, n_seqs,
                    max_new, nh, nkv, hd, page_size, chunk, window, scale, skip_single, sink, nullptr, key_splits,
                    part_acc, part_ml, status, 0, nullptr, 0, 0, softcap, slopes, sink_values, keep, nullptr, stream);
}

// Sigmoid weights with the result written by the kernel itself: `out` [n_tokens, nh, hd] bfloat16 takes every
// row's plain sum over ALL its keys, turned back by the row's position when the values are cached rotated
// (`v_inv_freq` [v_pairs] or null; without `v_interleaved` the pairs are (m, m + hd / 2) and v_pairs == hd / 2).
// Rows of requests that `skip_single` leaves out are not written.
extern "C" int hb_sigmoid_prefill_tc(const void* q, const void* k_pages, const void* v_pages, const int* block_table,
                                     int table_stride, const int* cu_seqlens, const int* positions, void* out,
                                     int n_tokens, int n_pages, int n_seqs, int max_new, int nh, int nkv, int hd,
                                     int page_size, int chunk, int window, float scale, int skip_single,
                                     const float* head_bias, const float* v_inv_freq, int v_pairs, int v_interleaved,
                                     int* status, cudaStream_t stream) {
  if (v_pairs < 0 || (v_pairs > 0 && !v_inv_freq) || 2 * v_pairs > hd) return HB_ERR_BAD_ARG;
  if (v_pairs > 0 && !v_interleaved && 2 * v_pairs != hd) return HB_ERR_UNSUPPORTED;
  return prefill_tc(q, k_pages, v_pages, block_table, table_stride, cu_seqlens, positions, out, n_tokens, n_pages, n_seqs,
                    max_new, nh, nkv, hd, page_size, chunk, window, scale, skip_single, 2, head_bias, 1, nullptr, nullptr,
                    status, 1, v_inv_freq, v_pairs, v_interleaved, 0.f, nullptr, nullptr, 0, nullptr, stream);
}

// Differential attention: q [n_tokens, nh, hd] holds the two maps of head a as heads 2a and 2a + 1, both over the same
// key and value rows of kv head 2a / (nh / nkv) (a map's query is zero where the row belongs to the other map's key).
// out [n_tokens, nh / 2, vdim] bfloat16 = (a1 - lambda a2) rsqrt(mean(.^2) + eps) mul, times sigmoid(gate) where
// `gate` (bfloat16, row t at gate + t * gate_stride, nh / 2 * vdim wide) is given. Rows of requests that `skip_single`
// leaves out are not written.
extern "C" int hb_diff_prefill_tc(const void* q, const void* k_pages, const void* v_pages, const int* block_table,
                                  int table_stride, const int* cu_seqlens, const int* positions, void* out, int n_tokens,
                                  int n_pages, int n_seqs, int max_new, int nh, int nkv, int hd, int page_size, int chunk,
                                  int window, int keep, float scale, int skip_single, float lambda, float eps, float mul,
                                  int vdim, const void* gate, long long gate_stride, int* status, cudaStream_t stream) {
  if (nh % 2 != 0 || nkv <= 0 || (nh / nkv) % 2 != 0 || vdim <= 0 || vdim > hd || (gate && gate_stride < (long long)(nh / 2) * vdim))
    return HB_ERR_BAD_ARG;
  const bool vec = vdim % 8 == 0 && ((uintptr_t)out & 15) == 0 && (!gate || (((uintptr_t)gate & 15) == 0 && gate_stride % 8 == 0));
  const Pair pair{lambda, eps, mul, vdim, vec ? 1 : 0, (const __nv_bfloat16*)gate, gate_stride};
  return prefill_tc(q, k_pages, v_pages, block_table, table_stride, cu_seqlens, positions, out, n_tokens, n_pages, n_seqs,
                    max_new, nh, nkv, hd, page_size, chunk, window, scale, skip_single, 0, nullptr, 1, nullptr, nullptr,
                    status, 0, nullptr, 0, 0, 0.f, nullptr, nullptr, keep, &pair, stream);
}

namespace {
int prefill_tc(const void* q, const void* k_pages, const void* v_pages, const int* block_table, int table_stride,
               const int* cu_seqlens, const int* positions, void* out, int n_tokens, int n_pages, int n_seqs, int max_new,
               int nh, int nkv, int hd, int page_size, int chunk, int window, float scale, int skip_single, int sink,
               const float* head_bias, int key_splits, float* part_acc, float* part_ml, int* status, int turn_inside,
               const float* v_inv_freq, int v_pairs, int v_interleaved, float softcap, const float* slopes,
               const float* sink_values, int keep, const Pair* pair, cudaStream_t stream) {
  if (sink == 2 && (softcap > 0.f || slopes || sink_values)) return HB_ERR_UNSUPPORTED;
  if (!q || !k_pages || !v_pages || !block_table || !cu_seqlens || !positions || !out || !status) return HB_ERR_BAD_ARG;
  if (n_tokens < 0 || n_pages <= 0 || n_seqs < 0 || max_new < 0 || nh <= 0 || nkv <= 0 || nh % nkv != 0 ||
      page_size <= 0 || table_stride <= 0 || chunk < 0 || window < 0 || key_splits < 1 || key_splits > 64 ||
      keep < 0 || (keep > 0 && window <= 0) || (sink == 2 && !turn_inside ? !part_acc : (key_splits > 1 && (!part_acc || !part_ml))))
    return HB_ERR_BAD_ARG;
  if (keep > 0 && key_splits > 1) return HB_ERR_UNSUPPORTED;
  if (page_size % 16 != 0 || !(BKEYS % page_size == 0 || page_size % BKEYS == 0)) return HB_ERR_UNSUPPORTED;
  if (n_seqs > 65535 || nh > 65535) return HB_ERR_UNSUPPORTED;
  if (!(scale > 0.f)) return HB_ERR_UNSUPPORTED;       // the largest raw score is taken for the largest scaled one
  if (n_seqs == 0 || max_new == 0 || n_tokens == 0) return HB_OK;
  Args a{block_table, cu_seqlens, positions, (__nv_bfloat16*)out, status, table_stride, nh, nkv, page_size, chunk,
         window, skip_single, page_size < BKEYS ? page_size : BKEYS, scale * 1.4426950408889634f, key_splits, part_acc, part_ml, sink, head_bias,
         turn_inside, v_pairs, v_interleaved, v_inv_freq, softcap, slopes, sink_values, slopes ? 1 : 0, keep, pair ? *pair : Pair{}};
  const long long pool_rows = (long long)n_pages * nkv * page_size;
  if (pair) {
    if (hd == 192) return launch<192, true>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
    if (hd == 128) return launch<128, true>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
    if (hd == 64) return launch<64, true>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
    return HB_ERR_UNSUPPORTED;
  }
  if (hd == 192) return launch<192>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
  if (hd == 128) return launch<128>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
  if (hd == 64) return launch<64>(q, k_pages, v_pages, a, n_tokens, pool_rows, n_seqs, max_new, stream);
  return HB_ERR_UNSUPPORTED;
}
}  // namespace
