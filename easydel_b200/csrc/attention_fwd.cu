// Flash-attention forward on tcgen05 tensor cores (tiles of 64 or 128 columns per head, bf16, GQA,
// causal, variable-length batches, sliding window, logit soft-cap, attention sinks).
//
// The query / key size and the value size of a head are separate and may be any multiple of 8 up to 192 (keys) and 128
// (values): a tile is DQ (or DV) columns wide, 64, 128 or 192, and the tensor maps carry the real sizes, so the columns past a head's end
// arrive as zeros and only the real value columns are stored. Memory holds no padding.
//
// One CTA per (block of 256 query rows = two tiles A and B, query head, sequence):
//   warp 0      TMA producer: both Q tiles once, then K and V tiles of 128 keys through
//               two independent 2-stage rings (K is released as soon as both QK^T products
//               of a step are issued, V after both PV products)
//   warp 1      MMA issuer, software pipelined per key tile j:
//                   O_A += P_A(j) V(j);  S_A = Q_A K(j+1)^T;  O_B += P_B(j) V(j);  S_B = Q_B K(j+1)^T
//               so that the softmax of one tile always runs under the two products of the other
//   warps 2..9  softmax of tile A, warps 10..17 softmax of tile B. Two threads share a query row
//               (warps w and w + 4 of a group sit on the same tensor-memory lane quadrant and take
//               the left and the right 64 score columns): with one warp per scheduler the softmax of
//               a tile was bound by the latency of its own instruction stream and took longer than
//               the other tile's two products, which left the tensor pipe idle a fifth of the time.
//               Each thread pulls its 64 scores out of tensor memory, the two halves exchange their
//               maxima through shared memory, exponentiate in registers and write P back as packed
//               bf16 over the same tensor-memory columns (the A operand of the PV product). O is
//               rescaled in tensor memory only when the running maximum moved by more than 2^8.
// Weights without a softmax (ATT_SIGMOID: the sigmoid of score + a number per head, not normalised over keys) need neither
// maxima nor sums: the halves of a row never meet, and the output leaves times a gate per row.
// A window may keep the first tokens of a sequence: their key tiles come before the window's.
// Tensor memory map (512 columns): S_A/P_A [0,128)  S_B/P_B [128,256)  O_A [256,384)  O_B [384,512).
//
// Tiles 192 columns wide (expanded latent attention) leave shared memory for one stage of 128-wide values, and none for the
// exchange between the halves of a row: that goes through two spare tensor-memory columns of the row's own scores.
//
// Queries, keys and values are read straight out of the packed projection output
// through 3-D tensor maps (head_dim, heads, tokens), so no transposes are needed.
// The output and the log-sum-exp (for the backward pass) are written with plain
// predicated stores, which is what makes ragged sequence ends free.
//
// Takes the place of the cuDNN-FMHA / Triton flash kernels the reference reaches via
// easydel/operations/kernels/flash_attention.py:82-324 and
// scaled_dot_product_attention.py:107-254.
#include "common.cuh"
#include "tmem_ops.cuh"

#include <stdlib.h>

#include <type_traits>

namespace edl {
namespace {

constexpr int ATT_THREADS = 576;   // producer, MMA issuer, 2 x 8 softmax warps
constexpr int BQ = 128;
constexpr int BKV = 128;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float LN2 = 0.6931471805599453f;

// Optional cycle trace (-DEDL_ATTN_TRACE): CTA 0 stamps clock64 at the phase boundaries of its MMA-issuing lane and
// of one softmax thread per query tile, 64 steps x 8 slots per role; `edl_attn_trace_read` copies the table out
// (read by benchmarks/trace_attention.py).
#ifdef EDL_ATTN_TRACE
__device__ long long g_trace[4 * 64 * 8];
#define TRACE(role, n, slot) \
  do { if (trace_on && (n) < 64) g_trace[((role) * 64 + (n)) * 8 + (slot)] = clock64(); } while (0)
#else
#define TRACE(role, n, slot) do { } while (0)
#endif

struct AttnFwdParams {
  __nv_bfloat16* o;      // [tokens, ldo], head h at columns h*D
  long long ldo;
  float* lse;            // [Hq, total_q] natural-log sum-exp of the scaled scores
  const int* cu_q;       // [B+1] sequence starts in the token dimension, or null
  const int* cu_k;
  const float* sinks;    // [Hq] or null
  int B, Tq, Tk, Hq, Hkv, total_q;
  float scale_log2;      // softmax scale * log2(e)
  float softcap;         // 0 = off (applied to scaled scores, in natural units)
  int causal;
  int window;            // 0 = off; keys with pos <= qpos - window are masked
  int* status;
  // paged / packed mode (serving): keys and values live in pages of BKV tokens addressed through a
  // per-sequence page table, and the `pack` query heads of one KV head share a tile (row = token*pack + head)
  const int* page_table; // [B, pt_stride] page ids, or null
  const int* kv_lens;    // [B] keys per sequence (context length including the new tokens), paged mode
  int pt_stride;
  int pack;              // query heads per tile row group (1 = one head per CTA)
  int dq, dv;            // real query / key and value sizes of a head (<= the tile widths)
  int keep_first;        // with a window: keys before this position stay visible
  const float* score_bias;      // [Hq], ATT_SIGMOID
  const __nv_bfloat16* gate;    // [total_q, ld_gate] or null: output rows times sigmoid(gate[token][head])
  long long ld_gate;
  float out_scale;       // ATT_SIGMOID: factor of the output
  int nx, ny;            // launch geometry: query blocks and heads (the grid itself is one-dimensional)
};

template <int DQ, int DV>
struct ACfg {
  static constexpr int QCH = DQ / 64;             // 128-byte chunks along a query / key head
  static constexpr int VCH = DV / 64;             // ... and along a value head
  static constexpr int Q_BYTES = BQ * DQ * 2;     // one query tile
  static constexpr int K_BYTES = BKV * DQ * 2;
  static constexpr int V_BYTES = BKV * DV * 2;
  static constexpr bool WIDE = DQ > 128;
  static constexpr int VS = WIDE && DV > 64 ? 1 : 2;      // value stages
  // Without the exchange of maxima nothing tells one half of a row that the other has read its scores, so each half's P
  // stays over its own scores (columns of a score tile where the right half's P starts).
  static constexpr int P_RIGHT_SIG = 64;
  static constexpr int OFF_K = 2 * Q_BYTES;
  static constexpr int OFF_V = OFF_K + 2 * K_BYTES;
  static constexpr int OFF_BAR = OFF_V + VS * V_BYTES;
  static constexpr int OFF_XCH = OFF_BAR + 256;   // float [tile][parity][half][row]: row maxima / sums of a half
  static constexpr int SMEM = OFF_XCH + (WIDE ? 0 : 2 * 2 * 2 * BQ * 4) + 1024;
  static_assert(SMEM <= 232448, "shared memory of one CTA");
};

struct TileRange {
  int lo, hi;  // key-tile indices [lo, hi) this query tile attends to
};

__device__ __forceinline__ TileRange tile_range(int q0, int tq, int len_q, int len_k, int off, int causal,
                                                int window) {
  // q0: first query token of the tile, tq: query tokens per tile
  TileRange r{0, 0};
  if (q0 >= len_q) return r;
  int kv_hi = len_k;
  if (causal) kv_hi = min(len_k, q0 + tq + off);
  int kv_lo = 0;
  if (window > 0) kv_lo = max(0, q0 + off - window + 1);
  if (kv_hi <= kv_lo) return r;
  r.lo = kv_lo / BKV;
  r.hi = (kv_hi + BKV - 1) / BKV;
  return r;
}

// What becomes of the scores; forms of their own, so that none carries another's registers.
enum { ATT_SOFTMAX = 0, ATT_CAPPED = 1, ATT_SIGMOID = 2 };

template <int DQ, int DV, int MODE>
__global__ void __launch_bounds__(ATT_THREADS, 1)
attn_fwd_kernel(const __grid_constant__ CUtensorMap tq, const __grid_constant__ CUtensorMap tk,
                const __grid_constant__ CUtensorMap tv, const AttnFwdParams p) {
  using C = ACfg<DQ, DV>;
  constexpr bool CAP = MODE == ATT_CAPPED, SIG = MODE == ATT_SIGMOID;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sQ = smem_u32(smem);
  const uint32_t sK0 = sQ + C::OFF_K;
  const uint32_t sV0 = sQ + C::OFF_V;
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::OFF_BAR);
  const uint32_t b_qfull = smem_u32(bars);
  const uint32_t b_kfull = b_qfull + 8;        // [2]
  const uint32_t b_vfull = b_kfull + 16;       // [2]
  const uint32_t b_kempty = b_vfull + 16;      // [2]
  const uint32_t b_vempty = b_kempty + 16;     // [2]
  const uint32_t b_sfull = b_vempty + 16;      // [2] per query tile
  const uint32_t b_pfull = b_sfull + 16;       // [2] per query tile
  const uint32_t b_ofinal = b_pfull + 16;      // [2] per query tile
  const uint32_t b_xch = smem_u32(bars + 16);  // [2 tiles][4 quadrants]: the two halves of a row block meet here
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 15);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // One-dimensional grid, query block slowest and reversed: blocks are handed to SMs in index order, so the
  // long (late) causal blocks of every head and sequence start first and the short ones fill the tail.
  const int per_qb = p.ny * p.B;
  const int qb = p.nx - 1 - (int)(blockIdx.x / per_qb);
  const int rem_id = (int)(blockIdx.x % per_qb);
  const int b = rem_id / p.ny;
  const int pack = p.pack;                       // power of two, divides BQ
  const int pshift = 31 - __clz(pack);
  const int TQ = BQ >> pshift;                   // query tokens per tile
  const int h_first = (rem_id % p.ny) * pack;    // first query head of this CTA's rows
  const int hk = h_first / (p.Hq / p.Hkv);       // their KV head (pack divides the group)

  const int q_start = p.cu_q ? p.cu_q[b] : b * p.Tq;
  const int k_start = p.page_table ? 0 : (p.cu_k ? p.cu_k[b] : b * p.Tk);
  const int len_q = p.cu_q ? p.cu_q[b + 1] - q_start : p.Tq;
  const int len_k = p.kv_lens ? p.kv_lens[b] : (p.cu_k ? p.cu_k[b + 1] - k_start : p.Tk);
  const int* pt = p.page_table ? p.page_table + (long long)b * p.pt_stride : nullptr;
  const int qblock0 = qb * 2 * TQ;
  if (qblock0 >= len_q) return;
  const int off = len_k - len_q;  // absolute key position of query token r is r + off

  const TileRange rgA = tile_range(qblock0, TQ, len_q, len_k, off, p.causal, p.window);
  const TileRange rgB = tile_range(qblock0 + TQ, TQ, len_q, len_k, off, p.causal, p.window);
  const bool anyA = rgA.hi > rgA.lo, anyB = rgB.hi > rgB.lo;
  int jmin = 0, jmax = 0;
  if (anyA && anyB) {
    jmin = min(rgA.lo, rgB.lo);
    jmax = max(rgA.hi, rgB.hi);
  } else if (anyA) {
    jmin = rgA.lo;
    jmax = rgA.hi;
  } else if (anyB) {
    jmin = rgB.lo;
    jmax = rgB.hi;
  }
  // Steps of the key loop: the kept tiles in front of the windows first (every query of this block sees them), then
  // [jmin, jmax). Step i works on tile tile_at(i); a tile between the windows' starts may be one of the kept ones.
  const int kept_tiles = p.window > 0 ? (p.keep_first + BKV - 1) / BKV : 0;
  const int front = min(kept_tiles, jmin);
  const int steps = jmax > jmin ? front + jmax - jmin : 0;
  auto tile_at = [&](int i) { return i < front ? i : jmin + i - front; };

  if (threadIdx.x == 0) {
    mbar_init(b_qfull, 1);
    for (int s = 0; s < 2; ++s) {
      mbar_init(b_kfull + 8 * s, 1);
      mbar_init(b_vfull + 8 * s, 1);
      mbar_init(b_kempty + 8 * s, 1);
      mbar_init(b_vempty + 8 * s, 1);
      mbar_init(b_sfull + 8 * s, 1);
      mbar_init(b_pfull + 8 * s, 256);
      mbar_init(b_ofinal + 8 * s, 1);
    }
    for (int i = 0; i < 8; ++i) mbar_init(b_xch + 8 * i, 64);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(tmem_slot), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0) {
    if (lane == 0 && jmax > jmin) {
      prefetch_tmap(&tq);
      prefetch_tmap(&tk);
      prefetch_tmap(&tv);
      mbar_expect_tx(b_qfull, 2 * C::Q_BYTES);
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int c = 0; c < C::QCH; ++c)
          tma_load_3d(sQ + t * C::Q_BYTES + c * (BQ * 128), &tq, b_qfull, c * 64, h_first, q_start + qblock0 + t * TQ);
      auto row_of = [&](int j) { return pt ? pt[j] * BKV : k_start + j * BKV; };
      auto load_k = [&](int it) -> bool {
        const int s = it & 1, row = row_of(tile_at(it));
        if (it >= 2 &&
            !mbar_wait(b_kempty + 8 * s, ((it >> 1) - 1) & 1, abort_flag, p.status, EDL_TIMEOUT_PRODUCER))
          return false;
        mbar_expect_tx(b_kfull + 8 * s, C::K_BYTES);
#pragma unroll
        for (int c = 0; c < C::QCH; ++c)
          tma_load_3d(sK0 + s * C::K_BYTES + c * (BKV * 128), &tk, b_kfull + 8 * s, c * 64, hk, row);
        return true;
      };
      auto load_v = [&](int it) -> bool {
        const int s = it % C::VS, row = row_of(tile_at(it));
        if (it >= C::VS &&
            !mbar_wait(b_vempty + 8 * s, (it / C::VS - 1) & 1, abort_flag, p.status, EDL_TIMEOUT_PRODUCER))
          return false;
        mbar_expect_tx(b_vfull + 8 * s, C::V_BYTES);
#pragma unroll
        for (int c = 0; c < C::VCH; ++c)
          tma_load_3d(sV0 + s * C::V_BYTES + c * (BKV * 128), &tv, b_vfull + 8 * s, c * 64, hk, row);
        return true;
      };
      if constexpr (C::VS == 2) {
        for (int i = 0; i < steps; ++i)
          if (!load_k(i) || !load_v(i)) break;
      } else {   // the only value stage is free late: keys stay one tile ahead of it
        bool ok = load_k(0);
        for (int i = 0; i < steps && ok; ++i) ok = (i + 1 >= steps || load_k(i + 1)) && load_v(i);
      }
    }
  } else if (warp == 1) {
    if (jmax > jmin) {
      // The whole warp runs the role (waits, loop control, descriptor arithmetic); one elected lane issues.
      const bool leader = elect_one();
#ifdef EDL_ATTN_TRACE
      const bool trace_on = blockIdx.x == 0 && leader;
#endif
      constexpr uint32_t idesc_qk = umma_idesc_bf16(BQ, BKV, 0, 0);
      constexpr uint32_t idesc_pv = umma_idesc_bf16(BQ, DV, 0, 1);
      bool ok = mbar_wait(b_qfull, 0, abort_flag, p.status, EDL_TIMEOUT_MMA);
      int pv_cnt[2] = {0, 0};
      auto valid = [&](int t, int i) {
        const int j = tile_at(i);
        return t == 0 ? anyA && (j >= rgA.lo || j < kept_tiles) && j < rgA.hi
                      : anyB && (j >= rgB.lo || j < kept_tiles) && j < rgB.hi;
      };
      auto issue_qk = [&](int t, int i) {
        const int s = i & 1;
        const uint32_t kb = sK0 + s * C::K_BYTES;
        const uint32_t qbase = sQ + t * C::Q_BYTES;
#pragma unroll
        for (int c = 0; c < C::QCH; ++c)
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            uint64_t ad = umma_smem_desc_sw128(qbase + c * (BQ * 128) + k * 32, 16, 1024);
            uint64_t bd = umma_smem_desc_sw128(kb + c * (BKV * 128) + k * 32, 16, 1024);
            if (leader) umma_f16_ss(tmem_base + t * 128, ad, bd, idesc_qk, (c | k) != 0 ? 1u : 0u);
          }
        if (leader) tc_commit(b_sfull + 8 * t);
      };
      auto issue_pv = [&](int t, int i) -> bool {
        const int j = tile_at(i), s = i % C::VS;
        if (!mbar_wait(b_pfull + 8 * t, pv_cnt[t] & 1, abort_flag, p.status, EDL_TIMEOUT_MMA)) return false;
        tc_fence_after();
        const uint32_t vb = sV0 + s * C::V_BYTES;
#pragma unroll
        for (int k = 0; k < BKV / 16; ++k) {
          const int pc = SIG && k >= 4 ? C::P_RIGHT_SIG + (k - 4) * 8 : k * 8;
          uint64_t bd = umma_smem_desc_sw128(vb + k * 2048, BKV * 128, 1024);
          if (leader)
            umma_f16_ts(tmem_base + 256 + t * 128, tmem_base + t * 128 + pc, bd, idesc_pv,
                        (pv_cnt[t] | k) != 0 ? 1u : 0u);
        }
        ++pv_cnt[t];
        const bool last = t == 0 ? (j == rgA.hi - 1) : (j == rgB.hi - 1);
        if (last && leader) tc_commit(b_ofinal + 8 * t);
        return true;
      };
      if (ok) {
        ok = mbar_wait(b_kfull, 0, abort_flag, p.status, EDL_TIMEOUT_MMA);
        if (ok) {
          tc_fence_after();
          TRACE(3, 0, 0);
          if (valid(0, 0)) issue_qk(0, 0);
          TRACE(3, 0, 1);
          if (valid(1, 0)) issue_qk(1, 0);
          TRACE(3, 0, 2);
          if (leader) tc_commit(b_kempty);
        }
      }
      for (int it = 0; it < steps && ok; ++it) {
        const int s = it & 1;
        const bool more = it + 1 < steps;
        TRACE(2, it, 0);
        const int vs = it % C::VS;
        if (!mbar_wait(b_vfull + 8 * vs, (it / C::VS) & 1, abort_flag, p.status, EDL_TIMEOUT_MMA)) break;
        if (more && !mbar_wait(b_kfull + 8 * (s ^ 1), ((it + 1) >> 1) & 1, abort_flag, p.status, EDL_TIMEOUT_MMA))
          break;
        tc_fence_after();
        TRACE(2, it, 1);
        if (valid(0, it) && !issue_pv(0, it)) break;
        TRACE(2, it, 2);
        if (more && valid(0, it + 1)) issue_qk(0, it + 1);
        TRACE(2, it, 3);
        if (valid(1, it) && !issue_pv(1, it)) break;
        TRACE(2, it, 4);
        if (leader) tc_commit(b_vempty + 8 * vs);
        if (more) {
          if (valid(1, it + 1)) issue_qk(1, it + 1);
          if (leader) tc_commit(b_kempty + 8 * (s ^ 1));
        }
        TRACE(2, it, 5);
      }
    }
  } else {
    const int t = (warp - 2) >> 3;          // query tile handled by this softmax group
    const int half = ((warp - 2) >> 2) & 1; // score columns [64 * half, 64 * half + 64) of every key tile
    const int q = warp & 3;                 // tensor-memory lane quadrant of this warp
    const int r = q * 32 + lane;            // query row within the tile
    const int q0 = qblock0 + t * TQ;        // first query token of the tile
    const int qrow = q0 + (r >> pshift);    // query token (within the sequence) of this row
    const int qhead = h_first + (r & (pack - 1));
    const int qpos = qrow + off;            // absolute key position of this query
    const TileRange rg = t == 0 ? rgA : rgB;
    const uint32_t lane_sel = uint32_t(q * 32) << 16;
    const uint32_t tS = tmem_base + t * 128 + lane_sel;
    const uint32_t tO = tmem_base + 256 + t * 128 + lane_sel;
    const uint32_t bs = b_sfull + 8 * t, bp = b_pfull + 8 * t, bo = b_ofinal + 8 * t;
    const uint32_t bx = b_xch + 8 * (t * 4 + q);
    float* xch = reinterpret_cast<float*>(smem + C::OFF_XCH) + t * (2 * 2 * BQ);   // [parity][half][row]
    float m_used = -1e30f;
    float l = 0.f;                          // sum over this thread's columns only
    const float cap2 = p.softcap * LOG2E;   // soft-cap in log2 units
    const float cap_k2 = CAP ? 2.f * p.scale_log2 / p.softcap : 0.f;
    const float cap_k = cap_k2 * (0.5f * LN2);      // scale / cap
    const SoftCapNear near_cap(cap_k, cap2);
    const float mul = CAP ? 1.f : p.scale_log2;
    // sigmoid(score + bias) = 1 / (1 + 2^y), y = -(score + bias) log2 e
    const float sig_mul = SIG ? -p.scale_log2 : 0.f, sig_add = SIG ? -p.score_bias[qhead] * LOG2E : 0.f;
    bool alive = true;
    int n = 0;
    // One value per thread to the other half of the row and back (64-thread barrier, bounded). Wide tiles pass it through
    // tensor memory: the left half's value lies in a score column that the left half has read and that only the right
    // half overwrites (with its P, after reading it); the right half's in its own first column, which P never reaches.
    // At the end (`last`) P may still be an operand, so both use columns behind it, whose scores everyone has read
    // (not those of the step before, which the other half may still be reading).
    auto exchange = [&](float mine, float& other, bool last) -> bool {
      const int par = n & 1;
      if constexpr (C::WIDE) {
        const uint32_t left = tS + (last ? 65 : 63), right = tS + (last ? 66 : 64);
        tmem_st_32x32b_x1(half ? right : left, __float_as_uint(mine));
        tc_wait_st();
        tc_fence_before();
        mbar_arrive(bx);
        if (!mbar_wait(bx, par, abort_flag, p.status, EDL_TIMEOUT_SOFTMAX)) return false;
        tc_fence_after();
        uint32_t got;
        tmem_ld_32x32b_x1(half ? left : right, got);
        tc_wait_ld();
        other = __uint_as_float(got);
        return true;
      }
      xch[(par * 2 + half) * BQ + r] = mine;
      mbar_arrive(bx);
      if (!mbar_wait(bx, par, abort_flag, p.status, EDL_TIMEOUT_SOFTMAX)) return false;
      other = xch[(par * 2 + (half ^ 1)) * BQ + r];
      return true;
    };
#ifdef EDL_ATTN_TRACE
    const bool trace_on = blockIdx.x == 0 && q == 0 && lane == 0 && half == 0;
#endif
    const bool any = rg.hi > rg.lo;
    for (int it = 0; it < steps && alive; ++it) {
      const int j = tile_at(it);
      if (!any || j >= rg.hi || (j < rg.lo && j >= kept_tiles)) continue;      // not a tile of this group's
      const int kv0 = j * BKV;
      const int kbase = kv0 + half * 64;
      TRACE(t, n, 0);
      if (!mbar_wait(bs, n & 1, abort_flag, p.status, EDL_TIMEOUT_SOFTMAX)) {
        alive = false;
        break;
      }
      tc_fence_after();
      TRACE(t, n, 1);
      uint32_t a[64];
      tmem_ld_32x32b_x64(tS + half * 64, a);
      const bool tile_mask = (kv0 + BKV > len_k) || (p.causal && kv0 + BKV - 1 > q0 + off) ||
                             (p.window > 0 && kv0 < q0 + TQ - 1 + off - p.window + 1);
      tc_wait_ld();
      // Scores far below the cap in tiles without a mask stay raw: the cap is monotone, so the maximum is taken first, and
      // the polynomial goes into the exponents below. Elsewhere scores are capped here. Warp-uniform.
      bool raw = false;
      if constexpr (CAP) {
        float m0 = 0.f, m1 = 0.f;
#pragma unroll
        for (int i = 0; i < 64; i += 4) {
          m0 = fmax3(m0, fabsf(__uint_as_float(a[i])), fabsf(__uint_as_float(a[i + 1])));
          m1 = fmax3(m1, fabsf(__uint_as_float(a[i + 2])), fabsf(__uint_as_float(a[i + 3])));
        }
        const float y = fmaxf(m0, m1) * cap_k;
        raw = __all_sync(0xffffffffu, y <= SOFT_CAP_NEAR_MAX) && !tile_mask;
        if (raw) {
        } else if (__all_sync(0xffffffffu, y <= SOFT_CAP_POLY_MAX)) {   // no MUFU
#pragma unroll
          for (int i = 0; i < 64; i += 2) {
            float s0 = __uint_as_float(a[i]), s1 = __uint_as_float(a[i + 1]);
            soft_cap_poly2(s0, s1, cap_k, cap2);
            a[i] = __float_as_uint(s0);
            a[i + 1] = __float_as_uint(s1);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 64; ++i) a[i] = __float_as_uint(soft_cap(__uint_as_float(a[i]), cap_k2, cap2));
        }
      }
      if (tile_mask) {
#pragma unroll
        for (int i = 0; i < 64; ++i) {
          const int k0 = kbase + i;
          const bool ok0 = (k0 < len_k) && (!p.causal || k0 <= qpos) &&
                           (p.window <= 0 || k0 > qpos - p.window || k0 < p.keep_first);
          if (!ok0) a[i] = 0xff800000u;  // -inf
        }
      }
      if constexpr (SIG) {
        // Four weights per step: two exponentials on the MUFU, two polynomials, and two reciprocals for the four of them
        // (1/x = y / (x y); y is bounded so that no product overflows, the weights it cuts off are below 2^-60).
        uint32_t pk[32];
        auto weights = [&](auto masked) {
#pragma unroll
          for (int i = 0; i < 64; i += 4) {
            float y0, y1, y2, y3;
            fma2(y0, y1, __uint_as_float(a[i]), __uint_as_float(a[i + 1]), sig_mul, sig_mul, sig_add, sig_add);
            fma2(y2, y3, __uint_as_float(a[i + 2]), __uint_as_float(a[i + 3]), sig_mul, sig_mul, sig_add, sig_add);
            const float d0 = 1.f + exp2f(fminf(y0, 60.f)), d1 = 1.f + exp2f(fminf(y1, 60.f));
            const float d2 = 1.f + exp2_poly(fminf(y2, 60.f)), d3 = 1.f + exp2_poly(fminf(y3, 60.f));
            const float r01 = __fdividef(1.f, d0 * d1), r23 = __fdividef(1.f, d2 * d3);
            float w0 = r01 * d1, w1 = r01 * d0, w2 = r23 * d3, w3 = r23 * d2;
            if constexpr (decltype(masked)::value) {
              if (a[i] == 0xff800000u) w0 = 0.f;
              if (a[i + 1] == 0xff800000u) w1 = 0.f;
              if (a[i + 2] == 0xff800000u) w2 = 0.f;
              if (a[i + 3] == 0xff800000u) w3 = 0.f;
            }
            pk[i >> 1] = pack_bf16x2(w0, w1);
            pk[(i >> 1) + 1] = pack_bf16x2(w2, w3);
          }
        };
        if (tile_mask) weights(std::true_type{}); else weights(std::false_type{});
        tmem_st_32x32b_x32(tS + half * C::P_RIGHT_SIG, pk);
        tc_wait_st();
        tc_fence_before();
        mbar_arrive(bp);
        ++n;
        continue;
      }
      float mx;
      {
        float m0 = fmax3(__uint_as_float(a[0]), __uint_as_float(a[1]), __uint_as_float(a[2]));
        float m1 = fmax3(__uint_as_float(a[3]), __uint_as_float(a[4]), __uint_as_float(a[5]));
#pragma unroll
        for (int i = 6; i < 62; i += 4) {
          m0 = fmax3(m0, __uint_as_float(a[i]), __uint_as_float(a[i + 1]));
          m1 = fmax3(m1, __uint_as_float(a[i + 2]), __uint_as_float(a[i + 3]));
        }
        mx = fmax3(m0, m1, fmaxf(__uint_as_float(a[62]), __uint_as_float(a[63])));
      }
      if (CAP && raw) mx = near_cap.at(mx);
      float mx_other;
      TRACE(t, n, 2);
      if (!exchange(mx, mx_other, false)) {
        alive = false;
        break;
      }
      mx = fmaxf(mx, mx_other) * mul;  // mul > 0, so scaling commutes with the maximum
      // lazy rescale. Both halves of a row see the same maxima, so they take the same decision (warp-uniform,
      // as tcgen05.ld/st are warp-wide) and each rescales its own half of O's columns. The QK^T product of this
      // step was issued after the PV product of the previous one, so O is quiescent here.
      const float m_new = fmaxf(m_used, mx);
      if (__any_sync(0xffffffffu, m_new > m_used + 8.f)) {
        const float alpha = exp2f(m_used - m_new);
        l *= alpha;
        if (n > 0) {
#pragma unroll 1
          for (int c = 0; c < DV / 64; ++c) {
            uint32_t rr[32];
            tmem_ld_32x32b_x32(tO + half * (DV / 2) + c * 32, rr);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) rr[i] = __float_as_uint(__uint_as_float(rr[i]) * alpha);
            tmem_st_32x32b_x32(tO + half * (DV / 2) + c * 32, rr);
          }
        }
        m_used = m_new;
      }
      const float neg_m = -m_used;
      TRACE(t, n, 3);
      float l0 = 0.f, l1 = 0.f, l2 = 0.f, l3 = 0.f;
      // Four scores per step: packed FMAs form x = s * mul - m, three exponentials go to the MUFU and one to the
      // polynomial on the FMA pipe, the row sum is accumulated with packed adds.
      uint32_t pk[32];
      auto exponentials = [&](auto argument) {
#pragma unroll
        for (int i = 0; i < 64; i += 4) {
          float x0, x1, x2, x3;
          argument(x0, x1, __uint_as_float(a[i]), __uint_as_float(a[i + 1]));
          argument(x2, x3, __uint_as_float(a[i + 2]), __uint_as_float(a[i + 3]));
          const float e0 = exp2f(x0), e1 = exp2f(x1), e2 = exp2f(x2);
          const float e3 = exp2_poly(x3);
          add2(l0, l1, e0, e1);
          add2(l2, l3, e2, e3);
          pk[i >> 1] = pack_bf16x2(e0, e1);
          pk[(i >> 1) + 1] = pack_bf16x2(e2, e3);
        }
      };
      if (CAP && raw)
        exponentials([&](float& x0, float& x1, float s0, float s1) { near_cap.add2(x0, x1, s0, s1, neg_m); });
      else
        exponentials([&](float& x0, float& x1, float s0, float s1) { fma2(x0, x1, s0, s1, mul, mul, neg_m, neg_m); });
      tmem_st_32x32b_x32(tS + half * 32, pk);
      l0 += l2;
      l1 += l3;
      l += l0 + l1;
      TRACE(t, n, 4);
      tc_wait_st();
      TRACE(t, n, 5);
      tc_fence_before();
      mbar_arrive(bp);
      TRACE(t, n, 6);
      ++n;
    }

    // epilogue: O / l -> bf16, plus LSE. Each half writes its own DV / 2 columns; the row sum is the two halves'.
    if (!SIG && any && alive) {
      float l_other;
      if (!exchange(l, l_other, true)) alive = false;
      l += l_other;
    }
    if (any && alive) {
      if (!mbar_wait(bo, 0, abort_flag, p.status, EDL_TIMEOUT_EPILOGUE)) alive = false;
      tc_fence_after();
    }
    if (alive && q0 < len_q) {
      const bool row_ok = qrow < len_q;
      float inv_l;
      if constexpr (SIG) {
        inv_l = p.out_scale;
        if (p.gate && row_ok) {
          const float g = __bfloat162float(p.gate[(long long)(q_start + qrow) * p.ld_gate + qhead]);
          inv_l = __fdividef(p.out_scale, 1.f + exp2f(fminf(-g * LOG2E, 60.f)));
        }
      } else {
        if (p.sinks) l += exp2f(p.sinks[qhead] * LOG2E - m_used);
        inv_l = l > 0.f ? 1.f / l : 0.f;
      }
      __nv_bfloat16* op = p.o + (long long)(q_start + qrow) * p.ldo + (long long)qhead * p.dv + half * (DV / 2);
#pragma unroll 1
      for (int c = 0; c < DV / 64; ++c) {
        uint32_t rr[32];
        if (any) {
          tmem_ld_32x32b_x32(tO + half * (DV / 2) + c * 32, rr);
          tc_wait_ld();
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i) rr[i] = 0u;
        }
        if (row_ok) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (half * (DV / 2) + c * 32 + i >= p.dv) break;   // dv is a multiple of 8
            uint4 o;
            o.x = pack_bf16x2(__uint_as_float(rr[i]) * inv_l, __uint_as_float(rr[i + 1]) * inv_l);
            o.y = pack_bf16x2(__uint_as_float(rr[i + 2]) * inv_l, __uint_as_float(rr[i + 3]) * inv_l);
            o.z = pack_bf16x2(__uint_as_float(rr[i + 4]) * inv_l, __uint_as_float(rr[i + 5]) * inv_l);
            o.w = pack_bf16x2(__uint_as_float(rr[i + 6]) * inv_l, __uint_as_float(rr[i + 7]) * inv_l);
            *reinterpret_cast<uint4*>(op + c * 32 + i) = o;
          }
        }
      }
      if (row_ok && p.lse && half == 0)
        p.lse[(long long)qhead * p.total_q + q_start + qrow] = l > 0.f ? (m_used + log2f(l)) * LN2 : -INFINITY;
    }
  }

  if (*abort_flag) {
    long long t0 = clock64();
    while (clock64() - t0 < 400000) {
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

template <int DQ, int DV, int MODE>
int launch_fwd_as(const void* q, const void* k, const void* v, long long ldq, long long ldk, long long ldv,
                  long long total_q, long long total_k, const AttnFwdParams& p, cudaStream_t stream) {
  using C = ACfg<DQ, DV>;
  CUtensorMap tq, tk, tv;
  if (make_tmap_3d_16b(&tq, q, p.dq, p.Hq, total_q, p.dq, ldq, 64, p.pack, BQ / p.pack, 3)) return -1;
  if (make_tmap_3d_16b(&tk, k, p.dq, p.Hkv, total_k, p.dq, ldk, 64, 1, BKV, 3)) return -1;
  if (make_tmap_3d_16b(&tv, v, p.dv, p.Hkv, total_k, p.dv, ldv, 64, 1, BKV, 3)) return -1;
  auto kern = attn_fwd_kernel<DQ, DV, MODE>;
  static bool attr_set[64] = {false};  // per device
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) dev = 0;
  if (!attr_set[dev]) {
    if (check_cuda(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM),
                   "cudaFuncSetAttribute(attn_fwd)"))
      return -1;
    attr_set[dev] = true;
  }
  const int tq_block = 2 * BQ / p.pack;  // query tokens per CTA
  AttnFwdParams pl = p;
  pl.nx = (p.Tq + tq_block - 1) / tq_block;
  pl.ny = p.Hq / p.pack;
  const long long blocks = (long long)pl.nx * pl.ny * p.B;
  kern<<<(unsigned)blocks, ATT_THREADS, C::SMEM, stream>>>(tq, tk, tv, pl);
  return check_cuda(cudaGetLastError(), "attn_fwd launch");
}

template <int DQ, int DV>
int launch_fwd(const void* q, const void* k, const void* v, long long ldq, long long ldk, long long ldv,
               long long total_q, long long total_k, const AttnFwdParams& p, cudaStream_t s) {
  if constexpr (DQ <= 128)
    if (p.score_bias) return launch_fwd_as<DQ, DV, ATT_SIGMOID>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s);
  return p.softcap > 0.f ? launch_fwd_as<DQ, DV, ATT_CAPPED>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s)
                         : launch_fwd_as<DQ, DV, ATT_SOFTMAX>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s);
}

// Tile widths from the real head sizes.
int dispatch_fwd(const void* q, const void* k, const void* v, long long ldq, long long ldk, long long ldv,
                 long long total_q, long long total_k, const AttnFwdParams& p, cudaStream_t s) {
  if (p.dq > 128)
    return p.dv > 64 ? launch_fwd<192, 128>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s)
                     : launch_fwd<192, 64>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s);
  if (p.dq > 64)
    return p.dv > 64 ? launch_fwd<128, 128>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s)
                     : launch_fwd<128, 64>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s);
  return p.dv > 64 ? launch_fwd<64, 128>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s)
                   : launch_fwd<64, 64>(q, k, v, ldq, ldk, ldv, total_q, total_k, p, s);
}

}  // namespace
}  // namespace edl

#ifdef EDL_ATTN_TRACE
EDL_HOST_API int edl_attn_trace_read(long long* host) {
  return (int)cudaMemcpyFromSymbol(host, edl::g_trace, sizeof(long long) * 4 * 64 * 8);
}
#endif

// q: [total_q, ldq] with head h at columns h*D (bf16); k, v likewise with Hkv heads.
// Fixed-length batches: cu_q = cu_k = null, total_q = B*Tq, total_k = B*Tk. Variable
// length: cu_q/cu_k are device int32[B+1] prefix sums and Tq/Tk the maximum lengths.
// Queries are aligned to the end of the keys (query row r sits at key position
// r + len_k - len_q). o: [total_q, ldo]; lse: [Hq, total_q] fp32 (may be null).
EDL_HOST_API int edl_attn_fwd(const void* q, const void* k, const void* v, void* o, float* lse, long long ldq,
                              long long ldk, long long ldv, long long ldo, const int* cu_q, const int* cu_k, int B,
                              int Tq, int Tk, long long total_q, long long total_k, int Hq, int Hkv, int D,
                              float scale, int causal, int window, float softcap, const float* sinks, int* status,
                              void* stream) {
  using namespace edl;
  if (B <= 0 || Tq <= 0 || total_q <= 0) return 0;
  if (D != 64 && D != 128) {
    set_last_error("edl_attn_fwd: head_dim %d not supported (64 or 128)", D);
    return -1;
  }
  if (Hq % Hkv) {
    set_last_error("edl_attn_fwd: Hq=%d not a multiple of Hkv=%d", Hq, Hkv);
    return -1;
  }
  if ((ldo & 7) || (reinterpret_cast<uintptr_t>(o) & 15)) {
    set_last_error("edl_attn_fwd: output must be 16-byte aligned with ldo %% 8 == 0");
    return -1;
  }
  AttnFwdParams p;
  p.o = reinterpret_cast<__nv_bfloat16*>(o);
  p.ldo = ldo;
  p.lse = lse;
  p.cu_q = cu_q;
  p.cu_k = cu_k;
  p.sinks = sinks;
  p.B = B;
  p.Tq = Tq;
  p.Tk = Tk;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.total_q = (int)total_q;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.softcap = softcap;
  p.causal = causal;
  p.window = window;
  p.status = status;
  p.page_table = nullptr;
  p.kv_lens = nullptr;
  p.pt_stride = 0;
  p.pack = 1;
  p.dq = p.dv = D;
  p.keep_first = 0;
  p.score_bias = nullptr;
  p.gate = nullptr;
  p.ld_gate = 0;
  p.out_scale = 1.f;
  return dispatch_fwd(q, k, v, ldq, ldk, ldv, total_q, total_k, p, reinterpret_cast<cudaStream_t>(stream));
}

// Paged attention for serving (mixed prefill + decode in one launch).
//   q:        [total_q, ldq] new query tokens of all sequences, concatenated; cu_q [B+1] their offsets
//   k_pages / v_pages: [num_pages * 128, ld_kpage / ld_vpage] page pools (page size 128 tokens), heads packed in a row;
//             the new tokens' keys/values must already be written to their pages
//   page_table [B, pt_stride]: page ids of each sequence in order; kv_lens [B]: keys per sequence
//             (cached + new). Query token i of a sequence sits at key position kv_len - len_q + i.
//   max_q:    largest number of new tokens of any sequence (sizes the grid)
// All query heads of a KV head share one tile (rows = token x head), so one pass over a page
// serves the whole GQA group; a group whose size is not a power of two is cut into equal power-of-two parts.
// Head sizes: multiples of 8, D (queries, keys) up to 192 and Dv (values) up to 128.
static int attn_paged_impl(const void* q, const void* k_pages, const void* v_pages, void* o, float* lse,
                           long long ldq, long long ld_kpage, long long ld_vpage, long long ldo, const int* cu_q, const int* kv_lens,
                           const int* page_table, int pt_stride, int B, int max_q, long long total_q,
                           long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int causal, int window,
                           float softcap, const float* sinks, int* status, void* stream, int keep_first = 0,
                           const float* score_bias = nullptr, const void* gate = nullptr, long long ld_gate = 0,
                           float out_scale = 1.f) {
  using namespace edl;
  if (B <= 0 || max_q <= 0 || total_q <= 0) return 0;
  if (score_bias && (D > 128 || softcap > 0.f || sinks || lse)) {
    set_last_error("edl_attn_paged: sigmoid weights go with heads up to 128 wide and without cap, sinks and log-sum-exp");
    return -1;
  }
  if (D < 8 || D > 192 || (D & 7) || Dv < 8 || Dv > 128 || (Dv & 7) || Hkv < 1 || Hq % Hkv) {
    set_last_error("edl_attn_paged: unsupported head layout (D=%d, Dv=%d, Hq=%d, Hkv=%d)", D, Dv, Hq, Hkv);
    return -1;
  }
  const int group = Hq / Hkv;
  int G = group & -group;            // largest power of two that divides the group
  if (G > 128) G = 128;
  if ((ldo & 7) || (reinterpret_cast<uintptr_t>(o) & 15)) {
    set_last_error("edl_attn_paged: output must be 16-byte aligned with ldo %% 8 == 0");
    return -1;
  }
  AttnFwdParams p;
  p.o = reinterpret_cast<__nv_bfloat16*>(o);
  p.ldo = ldo;
  p.lse = lse;
  p.cu_q = cu_q;
  p.cu_k = nullptr;
  p.sinks = sinks;
  p.B = B;
  p.Tq = max_q;
  p.Tk = 0;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.total_q = (int)total_q;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.softcap = softcap;
  p.causal = causal;
  p.window = window;
  p.status = status;
  p.page_table = page_table;
  p.kv_lens = kv_lens;
  p.pt_stride = pt_stride;
  p.pack = G;
  p.dq = D;
  p.dv = Dv;
  p.keep_first = keep_first;
  p.score_bias = score_bias;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.ld_gate = ld_gate;
  p.out_scale = out_scale;
  return dispatch_fwd(q, k_pages, v_pages, ldq, ld_kpage, ld_vpage, total_q, num_pages * 128, p,
                      reinterpret_cast<cudaStream_t>(stream));
}

EDL_HOST_API int edl_attn_paged(const void* q, const void* k_pages, const void* v_pages, void* o, long long ldq,
                                long long ld_kpage, long long ld_vpage, long long ldo, const int* cu_q,
                                const int* kv_lens, const int* page_table, int pt_stride, int B, int max_q, long long total_q,
                                long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int causal, int window,
                                int keep_first, float softcap, const float* sinks, int* status, void* stream) {
  return attn_paged_impl(q, k_pages, v_pages, o, nullptr, ldq, ld_kpage, ld_vpage, ldo, cu_q, kv_lens, page_table, pt_stride, B,
                         max_q, total_q, num_pages, Hq, Hkv, D, Dv, scale, causal, window, softcap, sinks, status, stream,
                         keep_first);
}

// The same without a softmax: a visible key's weight is sigmoid(score + score_bias[head]); the output is multiplied by
// out_scale and, with a gate [total_q, ld_gate] (bf16), by sigmoid(gate[token][head]). D up to 128.
EDL_HOST_API int edl_attn_paged_sigmoid(const void* q, const void* k_pages, const void* v_pages, void* o, long long ldq,
                                        long long ld_kpage, long long ld_vpage, long long ldo, const int* cu_q,
                                        const int* kv_lens, const int* page_table, int pt_stride, int B, int max_q,
                                        long long total_q, long long num_pages, int Hq, int Hkv, int D, int Dv, float scale,
                                        int window, int keep_first, const float* score_bias, const void* gate,
                                        long long ld_gate, float out_scale, int* status, void* stream) {
  return attn_paged_impl(q, k_pages, v_pages, o, nullptr, ldq, ld_kpage, ld_vpage, ldo, cu_q, kv_lens, page_table, pt_stride, B,
                         max_q, total_q, num_pages, Hq, Hkv, D, Dv, scale, 1, window, 0.f, nullptr, status, stream, keep_first,
                         score_bias, gate, ld_gate, out_scale);
}

// Same, also writing lse [Hq, total_q] (natural log of the softmax denominator; -inf for a row without keys):
// the partial results of split-KV decode and of context-parallel attention are merged from (o, lse) pairs.
EDL_HOST_API int edl_attn_paged_lse(const void* q, const void* k_pages, const void* v_pages, void* o, float* lse,
                                    long long ldq, long long ld_kpage, long long ld_vpage, long long ldo, const int* cu_q,
                                    const int* kv_lens, const int* page_table, int pt_stride, int B, int max_q,
                                    long long total_q, long long num_pages, int Hq, int Hkv, int D, int Dv, float scale,
                                    int causal, int window, float softcap, const float* sinks, int* status,
                                    void* stream) {
  return attn_paged_impl(q, k_pages, v_pages, o, lse, ldq, ld_kpage, ld_vpage, ldo, cu_q, kv_lens, page_table, pt_stride, B,
                         max_q, total_q, num_pages, Hq, Hkv, D, Dv, scale, causal, window, softcap, sinks, status, stream);
}
