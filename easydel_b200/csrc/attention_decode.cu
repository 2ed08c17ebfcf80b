// Paged decode attention: one new query token per sequence, grouped-query heads, long key ranges.
//
// A decode step has almost no arithmetic per byte (the G query heads of one KV head share every key / value row
// they read), so the job is to keep as many page bytes in flight as HBM can deliver. The tcgen05 kernel of
// attention_fwd.cu processes a sequence as one 128-row tile with a two-stage ring and spends microseconds per
// 128-key step on a tile that holds G real rows; this kernel is the streaming form:
//
//   * one CTA per (sequence, KV head, key split); its four warps take 32-key tiles round-robin, each warp with its
//     own three-stage ring of [32 keys x D] K and V tiles filled by TMA (lane 0 issues, an mbarrier per stage
//     receives the bytes), so 4 x 2 x 16 KB are in flight per CTA without any CTA-wide synchronisation;
//   * scores and the weighted value sum run on the tensor cores as m16n8k16 bf16 products (the G <= 16 query rows
//     are the M side; the 5th-generation MMA path has no shape this small, and the kernel is bandwidth bound);
//   * every warp keeps an online softmax for its keys; at the end the four partial (max, sum, O) triples are merged
//     through shared memory and written as bf16 rows, plus the log-sum-exp when the caller merges key splits.
//
// Replaces the decode branch of the reference's ragged / paged attention kernels
// (easydel/operations/kernels/ragged_page_attention_v3.py, page_attention.py). Query / key and value sizes of a head are
// separate multiples of 8 up to 128: tiles are DQ / DV = 64 or 128 columns wide and the tensor maps fill the columns
// past a head's end with zeros.
#include "common.cuh"

namespace edl {
namespace {

#ifndef EDL_DEC_WARPS
#define EDL_DEC_WARPS 4
#endif
#ifndef EDL_DEC_TK
#define EDL_DEC_TK 32
#endif
constexpr int DEC_WARPS = EDL_DEC_WARPS;
constexpr int DEC_THREADS = DEC_WARPS * 32;
constexpr int TK = EDL_DEC_TK;        // keys per tile (16 or 32)
constexpr int DEC_STAGES = 3;
constexpr int PAGE = 128;
constexpr float LOG2E_F = 1.4426950408889634f;

struct DecodeParams {
  const __nv_bfloat16* q;   // [B, ldq]: head h at columns h * dq
  long long ldq;
  __nv_bfloat16* o;         // [splits, B, ldo]
  long long ldo;
  float* lse;               // [splits, Hq, B] natural log-sum-exp per output row, or null
  const int* kv_lens;       // [B]
  const int* page_table;    // [B, pt_stride]
  const float* sinks;       // [Hq] or null (only without splits)
  int pt_stride, B, Hq, Hkv, splits, window;
  int dq, dv;               // real query / key and value sizes of a head
  float scale_log2;
  float cap_k2, cap2;       // soft-cap (see soft_cap), cap2 = 0: none
  int* status;
  int keep_first;           // with a window: keys before this position stay visible
  const float* score_bias;  // [Hq]: no softmax, weights are sigmoid(score + bias) (SIG)
  const __nv_bfloat16* gate;   // [B, ld_gate] or null: output rows times sigmoid(gate[b][head]) (SIG)
  long long ld_gate;
  float out_scale;          // SIG
  float* parts;             // SIG with splits > 1: fp32 [splits, B, Hq, dv], the parts of a plain sum
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Byte offset of (row, 16-byte chunk) inside a [TK rows x D] tile stored as D/64 boxes of [TK x 128 bytes] with the
// 128-byte swizzle the tensor maps use (chunk index XOR row % 8 within a box).
__device__ __forceinline__ uint32_t tile_off(int row, int chunk) {
  const int box = chunk >> 3, c = chunk & 7;
  return box * (TK * 128) + row * 128 + ((c ^ (row & 7)) << 4);
}

template <int DQ, int DV>
struct DCfg {
  static constexpr int K_BYTES = TK * DQ * 2;                         // one K tile
  static constexpr int STAGE_BYTES = K_BYTES + TK * DV * 2;           // K + V
  static constexpr int WARP_BYTES = DEC_STAGES * STAGE_BYTES;
  static constexpr int Q_BYTES = 16 * (DQ * 2 + 16);                  // 16 rows, padded pitch against bank conflicts
  static constexpr int OFF_Q = DEC_WARPS * WARP_BYTES;
  static constexpr int OFF_BAR = OFF_Q + Q_BYTES;
  static constexpr int OFF_RED = OFF_BAR + 128;                       // merge area: per warp m[16], l[16]
  static constexpr int SMEM = OFF_RED + DEC_WARPS * 2 * 16 * 4 + 1024;
};

template <int DQ, int DV, bool SIG>
__global__ void __launch_bounds__(DEC_THREADS)
attn_decode_kernel(const __grid_constant__ CUtensorMap tk, const __grid_constant__ CUtensorMap tv,
                   const DecodeParams p) {
  using C = DCfg<DQ, DV>;
  constexpr int NKS = DQ / 16;     // k-steps of the score product
  constexpr int NDB = DV / 8;     // 8-column blocks of the output
  constexpr int QPITCH = DQ * 2 + 16;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sbase = smem_u32(smem);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = p.Hq / p.Hkv;

  const int split = blockIdx.x % p.splits;
  const int hk = (blockIdx.x / p.splits) % p.Hkv;
  const int b = blockIdx.x / (p.splits * p.Hkv);
  const int kv_len = p.kv_lens[b];
  const int* pt = p.page_table + (long long)b * p.pt_stride;

  // key range of this split, in 32-key tiles (whole tiles; the ragged end is masked)
  int lo = 0;
  if (p.window > 0) lo = max(0, kv_len - p.window);
  const int t_first = lo / TK, t_end = (kv_len + TK - 1) / TK;
  // kept tiles in front of the window come first: place v of the list is tile tile_at(v)
  const int front = p.window > 0 ? min((p.keep_first + TK - 1) / TK, t_first) : 0;
  auto tile_at = [&](int v) { return v < front ? v : t_first + v - front; };
  const int n_all = max(0, front + t_end - t_first);
  const int per_split = (n_all + p.splits - 1) / p.splits;
  const int t0 = split * per_split;
  const int t1 = min(n_all, t0 + per_split);
  const int n_tiles = max(0, t1 - t0);
  // places of this warp: t0 + warp, t0 + warp + 4, ...
  const int my_n = n_tiles > warp ? (n_tiles - warp + DEC_WARPS - 1) / DEC_WARPS : 0;

  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::OFF_BAR);
  const uint32_t my_bar0 = smem_u32(bars) + warp * DEC_STAGES * 8;
  const uint32_t my_ring = sbase + warp * C::WARP_BYTES;
  __shared__ int s_abort;
  if (threadIdx.x == 0) {
    for (int i = 0; i < DEC_WARPS * DEC_STAGES; ++i) mbar_init(smem_u32(bars) + 8 * i, 1);
    s_abort = 0;
    fence_mbar_init();
    prefetch_tmap(&tk);
    prefetch_tmap(&tv);
  }
  // query rows of this KV head's group -> shared memory (rows >= G and columns >= dq are zero)
  {
    const __nv_bfloat16* qrow = p.q + (long long)b * p.ldq + (long long)hk * G * p.dq;
    for (int i = threadIdx.x; i < 16 * (DQ / 8); i += DEC_THREADS) {
      const int r = i / (DQ / 8), c = i % (DQ / 8);
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < G && c * 8 < p.dq) v = *reinterpret_cast<const uint4*>(qrow + (long long)r * p.dq + c * 8);
      *reinterpret_cast<uint4*>(smem + C::OFF_Q + r * QPITCH + c * 16) = v;
    }
  }
  __syncthreads();
  volatile int* abort_flag = &s_abort;

  auto issue = [&](int i) {   // lane 0 only: tile i of this warp into stage i % DEC_STAGES
    const int tile = tile_at(t0 + warp + i * DEC_WARPS);
    const int page = pt[tile / (PAGE / TK)];
    const int row = page * PAGE + (tile % (PAGE / TK)) * TK;
    const int st = i % DEC_STAGES;
    const uint32_t bar = my_bar0 + 8 * st;
    const uint32_t dst = my_ring + st * C::STAGE_BYTES;
    mbar_expect_tx(bar, C::STAGE_BYTES);
#pragma unroll
    for (int c = 0; c < DQ / 64; ++c) tma_load_3d(dst + c * (TK * 128), &tk, bar, c * 64, hk, row);
#pragma unroll
    for (int c = 0; c < DV / 64; ++c)
      tma_load_3d(dst + C::K_BYTES + c * (TK * 128), &tv, bar, c * 64, hk, row);
  };
  if (lane == 0)
    for (int i = 0; i < min(my_n, DEC_STAGES - 1); ++i) issue(i);

  // A fragments of Q (16 rows x DQ), loaded once
  uint32_t qa[NKS][4];
  {
    const uint32_t qb = sbase + C::OFF_Q;
#pragma unroll
    for (int ks = 0; ks < NKS; ++ks) {
      // matrices: (rows 0-7, k 0-7), (rows 8-15, k 0-7), (rows 0-7, k 8-15), (rows 8-15, k 8-15) of this k-step
      const int r = (lane & 7) + ((lane >> 3) & 1) * 8;
      const int kc = ks * 2 + (lane >> 4);
      ldmatrix_x4(qb + r * QPITCH + kc * 16, qa[ks]);
    }
  }

  float o_acc[NDB][4];
#pragma unroll
  for (int j = 0; j < NDB; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o_acc[j][e] = 0.f;
  float m_run[2] = {-1e30f, -1e30f};   // rows lane/4 and lane/4 + 8
  float l_run[2] = {0.f, 0.f};
  bool alive = true;
  float bias2[2] = {0.f, 0.f};         // score bias of rows lane/4 and lane/4 + 8, in log2 units
  if constexpr (SIG) {
#pragma unroll
    for (int h = 0; h < 2; ++h)
      if ((lane >> 2) + h * 8 < G) bias2[h] = p.score_bias[hk * G + (lane >> 2) + h * 8] * LOG2E_F;
  }

  for (int i = 0; i < my_n && alive; ++i) {
    const int st = i % DEC_STAGES;
    if (lane == 0 && i + DEC_STAGES - 1 < my_n) issue(i + DEC_STAGES - 1);   // its stage was consumed at step i - 1
    if (!mbar_wait(my_bar0 + 8 * st, (i / DEC_STAGES) & 1, abort_flag, p.status, EDL_TIMEOUT_SOFTMAX)) {
      alive = false;
      break;
    }
    const uint32_t kt = my_ring + st * C::STAGE_BYTES;
    const uint32_t vt = kt + C::K_BYTES;
    const int tile = tile_at(t0 + warp + i * DEC_WARPS);
    const int key0 = tile * TK;

    // ---- S = Q K^T for 32 keys: four 8-key blocks
    float s[TK / 8][4];
#pragma unroll
    for (int j = 0; j < TK / 8; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < NKS; ks += 2) {
        // four matrices of key block j: d-chunks 2ks, 2ks+1 (k-step ks) and 2ks+2, 2ks+3 (k-step ks+1)
        uint32_t kb[4];
        const int row = j * 8 + (lane & 7);
        ldmatrix_x4(kt + tile_off(row, ks * 2 + (lane >> 3)), kb);
        mma_bf16_16816(s[j], qa[ks], kb[0], kb[1]);
        mma_bf16_16816(s[j], qa[ks + 1], kb[2], kb[3]);
      }
    }
    // ---- mask the ragged end / the window start, online softmax (log2 domain)
    const int cbase = key0 + (lane & 3) * 2;
    uint32_t pa[TK / 16][4];
    if constexpr (SIG) {
#pragma unroll
      for (int j = 0; j < TK / 8; ++j) {
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
          const int key = cbase + j * 8;
          const bool ok0 = key < kv_len && (key >= lo || key < p.keep_first);
          const bool ok1 = key + 1 < kv_len && (key + 1 >= lo || key + 1 < p.keep_first);
          // one reciprocal for two weights; the bound keeps the product finite, what it cuts off is below 2^-60
          const float d0 = 1.f + exp2f(fminf(-fmaf(s[j][e], p.scale_log2, bias2[e >> 1]), 60.f));
          const float d1 = 1.f + exp2f(fminf(-fmaf(s[j][e + 1], p.scale_log2, bias2[e >> 1]), 60.f));
          const float r = __fdividef(1.f, d0 * d1);
          s[j][e] = ok0 ? r * d1 : 0.f;
          s[j][e + 1] = ok1 ? r * d0 : 0.f;
        }
        pa[j >> 1][(j & 1) * 2] = pack_bf16x2(s[j][0], s[j][1]);
        pa[j >> 1][(j & 1) * 2 + 1] = pack_bf16x2(s[j][2], s[j][3]);
      }
    } else {
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < TK / 8; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int key = cbase + j * 8 + (e & 1);
          const bool ok = key < kv_len && (key >= lo || key < p.keep_first);
          const float z = p.cap2 > 0.f ? soft_cap(s[j][e], p.cap_k2, p.cap2) : s[j][e] * p.scale_log2;
          s[j][e] = ok ? z : -INFINITY;
          mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
        }
      }
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
      }
      float alpha[2];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float m_new = fmaxf(m_run[h], mx[h]);
        alpha[h] = exp2f(m_run[h] - m_new);
        m_run[h] = m_new;
        l_run[h] *= alpha[h];
      }
      float rs[2] = {0.f, 0.f};
#pragma unroll
      for (int j = 0; j < TK / 8; ++j) {
        const float e0 = exp2f(s[j][0] - m_run[0]), e1 = exp2f(s[j][1] - m_run[0]);
        const float e2 = exp2f(s[j][2] - m_run[1]), e3 = exp2f(s[j][3] - m_run[1]);
        rs[0] += e0 + e1;
        rs[1] += e2 + e3;
        // S accumulator layout = A operand layout of the next product: blocks 2t, 2t+1 form k-step t
        pa[j >> 1][(j & 1) * 2] = pack_bf16x2(e0, e1);
        pa[j >> 1][(j & 1) * 2 + 1] = pack_bf16x2(e2, e3);
      }
      l_run[0] += rs[0];
      l_run[1] += rs[1];
      // ---- O = O * alpha + P V
#pragma unroll
      for (int j = 0; j < NDB; ++j) {
        o_acc[j][0] *= alpha[0];
        o_acc[j][1] *= alpha[0];
        o_acc[j][2] *= alpha[1];
        o_acc[j][3] *= alpha[1];
      }
    }
#pragma unroll
    for (int t = 0; t < TK / 16; ++t) {
#pragma unroll
      for (int j = 0; j < NDB; j += 2) {
        // transposed loads: (keys 16t..+7, chunk j), (keys 16t+8..+15, chunk j), the same two for chunk j+1
        uint32_t vb[4];
        const int row = t * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
        ldmatrix_x4_trans(vt + tile_off(row, j + (lane >> 4)), vb);
        mma_bf16_16816(o_acc[j], pa[t], vb[0], vb[1]);
        mma_bf16_16816(o_acc[j + 1], pa[t], vb[2], vb[3]);
      }
    }
    __syncwarp();   // every lane has read this stage before lane 0 refills it two steps later
  }

  // the row sums live spread over the four lanes that share a row
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
  }

  // ---- merge the four warps: (m, l) through shared memory, O through the (now idle) tile rings
  float* red = reinterpret_cast<float*>(smem + C::OFF_RED);   // [warp][m 16 | l 16]
  const int r0 = lane >> 2;
  if ((lane & 3) == 0) {
    red[warp * 32 + r0] = m_run[0];
    red[warp * 32 + r0 + 8] = m_run[1];
    red[warp * 32 + 16 + r0] = l_run[0];
    red[warp * 32 + 16 + r0 + 8] = l_run[1];
  }
  __syncthreads();
  float m_all[2], l_all[2], w_mine[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = r0 + h * 8;
    float m = -1e30f;
    for (int w = 0; w < DEC_WARPS; ++w) m = fmaxf(m, red[w * 32 + r]);
    float l = 0.f;
    for (int w = 0; w < DEC_WARPS; ++w) l += red[w * 32 + 16 + r] * exp2f(red[w * 32 + r] - m);
    m_all[h] = m;
    l_all[h] = l;
    w_mine[h] = SIG ? 1.f : exp2f(m_run[h] - m);
  }
  // each warp scales its O by its weight and adds it into a shared fp32 [16 x DV] accumulator, one warp after another
  float* o_sh = reinterpret_cast<float*>(smem);   // 16 * DV * 4 bytes <= one warp's ring
  for (int w = 0; w < DEC_WARPS; ++w) {
    if (warp == w) {
#pragma unroll
      for (int j = 0; j < NDB; ++j) {
        const int col = j * 8 + (lane & 3) * 2;
        float2* lo2 = reinterpret_cast<float2*>(o_sh + r0 * DV + col);
        float2* hi2 = reinterpret_cast<float2*>(o_sh + (r0 + 8) * DV + col);
        float2 a = w == 0 ? make_float2(0.f, 0.f) : *lo2;
        float2 c = w == 0 ? make_float2(0.f, 0.f) : *hi2;
        a.x += o_acc[j][0] * w_mine[0];
        a.y += o_acc[j][1] * w_mine[0];
        c.x += o_acc[j][2] * w_mine[1];
        c.y += o_acc[j][3] * w_mine[1];
        *lo2 = a;
        *hi2 = c;
      }
    }
    __syncthreads();
  }
  // ---- write: G rows of dv bf16 (+ LSE). Row r <-> query head hk * G + r.
  const long long orow = (long long)split * p.B + b;   // split-major: the layout edl_attn_combine reads
  for (int i = threadIdx.x; i < G * (DV / 8); i += DEC_THREADS) {
    const int r = i / (DV / 8), c = i % (DV / 8);
    if (c * 8 >= p.dv) continue;
    float m = -1e30f, l = 0.f;
    for (int w = 0; w < DEC_WARPS; ++w) m = fmaxf(m, red[w * 32 + r]);
    for (int w = 0; w < DEC_WARPS; ++w) l += red[w * 32 + 16 + r] * exp2f(red[w * 32 + r] - m);
    const int head = hk * G + r;
    if constexpr (SIG) {
      float f = p.out_scale;
      if (p.gate) {
        const float g = __bfloat162float(p.gate[(long long)b * p.ld_gate + head]);
        f = __fdividef(f, 1.f + exp2f(fminf(-g * LOG2E_F, 120.f)));
      }
      const float* src = o_sh + r * DV + c * 8;
      if (p.splits > 1) {
        float4* dst = reinterpret_cast<float4*>(p.parts + (orow * p.Hq + head) * p.dv + c * 8);
        dst[0] = make_float4(src[0] * f, src[1] * f, src[2] * f, src[3] * f);
        dst[1] = make_float4(src[4] * f, src[5] * f, src[6] * f, src[7] * f);
      } else {
        uint4 v;
        v.x = pack_bf16x2(src[0] * f, src[1] * f);
        v.y = pack_bf16x2(src[2] * f, src[3] * f);
        v.z = pack_bf16x2(src[4] * f, src[5] * f);
        v.w = pack_bf16x2(src[6] * f, src[7] * f);
        *reinterpret_cast<uint4*>(p.o + orow * p.ldo + (long long)head * p.dv + c * 8) = v;
      }
      continue;
    }
    if (p.sinks && p.splits == 1) l += exp2f(p.sinks[head] * LOG2E_F - m);
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const float* src = o_sh + r * DV + c * 8;
    uint4 v;
    v.x = pack_bf16x2(src[0] * inv, src[1] * inv);
    v.y = pack_bf16x2(src[2] * inv, src[3] * inv);
    v.z = pack_bf16x2(src[4] * inv, src[5] * inv);
    v.w = pack_bf16x2(src[6] * inv, src[7] * inv);
    *reinterpret_cast<uint4*>(p.o + orow * p.ldo + (long long)head * p.dv + c * 8) = v;
    if (c == 0 && p.lse)
      p.lse[((long long)split * p.Hq + head) * p.B + b] = l > 0.f ? (m + log2f(l)) * 0.6931471805599453f : -INFINITY;
  }
  (void)m_all;
  (void)l_all;
  if (s_abort) {   // a wait ran out: give copies still in flight time to land before shared memory is released
    long long t0c = clock64();
    while (clock64() - t0c < 400000) {
    }
  }
}

// out [B, width] (pitch ldo) = sum of the fp32 parts [splits, B, width]; width is a multiple of 8.
__global__ void sum_parts_kernel(const float* __restrict__ parts, int splits, int B, int width, __nv_bfloat16* __restrict__ out,
                                 long long ldo) {
  const long long total = (long long)B * (width / 4);
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int b = (int)(i / (width / 4)), c = (int)(i - (long long)b * (width / 4)) * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float4 v = *reinterpret_cast<const float4*>(parts + ((long long)s * B + b) * width + c);
      a.x += v.x;
      a.y += v.y;
      a.z += v.z;
      a.w += v.w;
    }
    *reinterpret_cast<uint2*>(out + b * ldo + c) = make_uint2(pack_bf16x2(a.x, a.y), pack_bf16x2(a.z, a.w));
  }
}

template <int DQ, int DV, bool SIG>
int launch_decode(const void* k_pages, const void* v_pages, long long ld_kpage, long long ld_vpage,
                  long long num_pages, const DecodeParams& p, cudaStream_t stream) {
  using C = DCfg<DQ, DV>;
  CUtensorMap tk, tv;
  const long long total_k = num_pages * PAGE;
  if (make_tmap_3d_16b(&tk, k_pages, p.dq, p.Hkv, total_k, p.dq, ld_kpage, 64, 1, TK, 3)) return -1;
  if (make_tmap_3d_16b(&tv, v_pages, p.dv, p.Hkv, total_k, p.dv, ld_vpage, 64, 1, TK, 3)) return -1;
  auto kern = attn_decode_kernel<DQ, DV, SIG>;
  static bool attr_set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) dev = 0;
  if (!attr_set[dev]) {
    if (check_cuda(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM),
                   "cudaFuncSetAttribute(attn_decode)"))
      return -1;
    attr_set[dev] = true;
  }
  const long long blocks = (long long)p.B * p.Hkv * p.splits;
  kern<<<(unsigned)blocks, DEC_THREADS, C::SMEM, stream>>>(tk, tv, p);
  if (SIG && p.splits > 1) {
    const int width = p.Hq * p.dv;
    const long long n = (long long)p.B * (width / 4);
    sum_parts_kernel<<<(int)((n + 255) / 256), 256, 0, stream>>>(p.parts, p.splits, p.B, width, p.o, p.ldo);
  }
  return check_cuda(cudaGetLastError(), "attn_decode launch");
}

template <bool SIG>
int dispatch_decode(const void* k_pages, const void* v_pages, long long ld_kpage, long long ld_vpage, long long num_pages,
                    const DecodeParams& p, cudaStream_t s) {
  if (p.dq > 64)
    return p.dv > 64 ? launch_decode<128, 128, SIG>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s)
                     : launch_decode<128, 64, SIG>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s);
  return p.dv > 64 ? launch_decode<64, 128, SIG>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s)
                   : launch_decode<64, 64, SIG>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s);
}

}  // namespace
}  // namespace edl

// Decode attention over a paged KV cache: q [B, ldq] (one token per sequence, head h at columns h * D),
// pages [num_pages * 128, ld_kpage / ld_vpage] with the KV heads packed in a row, page_table [B, pt_stride], kv_lens [B]
// (keys per sequence, the new token included). o [splits, B, ldo]; with splits > 1 part s holds the result over
// the s-th part of every sequence's keys and lse [splits, Hq, B] its log-sum-exp, for edl_attn_combine.
// Hq / Hkv <= 16; D (queries, keys) and Dv (values) are multiples of 8 up to 128; window = 0 or the sliding-window length,
// under which the first keep_first keys stay visible; softcap > 0: scores become softcap * tanh(scale * dot / softcap).
static int decode_impl(const void* q, const void* k_pages, const void* v_pages, void* o, float* lse,
                       long long ldq, long long ld_kpage, long long ld_vpage, long long ldo, const int* kv_lens,
                       const int* page_table, int pt_stride, int B, long long num_pages, int Hq, int Hkv,
                       int D, int Dv, float scale, int window, int keep_first, int splits, float softcap,
                       const float* sinks, const float* score_bias, const void* gate, long long ld_gate, float out_scale,
                       float* parts, int* status, void* stream) {
  using namespace edl;
  if (B <= 0) return 0;
  if (D < 8 || D > 128 || (D & 7) || Dv < 8 || Dv > 128 || (Dv & 7) || Hkv < 1 || Hq % Hkv || Hq / Hkv > 16 ||
      splits < 1) {
    set_last_error("edl_attn_decode: unsupported layout (D=%d, Dv=%d, Hq=%d, Hkv=%d, splits=%d)", D, Dv, Hq, Hkv,
                   splits);
    return -1;
  }
  if ((ldq & 7) || (ldo & 7) || (reinterpret_cast<uintptr_t>(q) & 15) || (reinterpret_cast<uintptr_t>(o) & 15)) {
    set_last_error("edl_attn_decode: q / o must be 16-byte aligned with row pitches that are multiples of 8");
    return -1;
  }
  DecodeParams p;
  p.q = reinterpret_cast<const __nv_bfloat16*>(q);
  p.ldq = ldq;
  p.o = reinterpret_cast<__nv_bfloat16*>(o);
  p.ldo = ldo;
  p.lse = lse;
  p.kv_lens = kv_lens;
  p.page_table = page_table;
  p.sinks = sinks;
  p.pt_stride = pt_stride;
  p.B = B;
  p.Hq = Hq;
  p.Hkv = Hkv;
  p.splits = splits;
  p.window = window;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.cap2 = softcap > 0.f ? softcap * 1.4426950408889634f : 0.f;
  p.cap_k2 = softcap > 0.f ? 2.f * p.scale_log2 / softcap : 0.f;
  p.status = status;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  p.dq = D;
  p.dv = Dv;
  p.keep_first = keep_first;
  p.score_bias = score_bias;
  p.gate = reinterpret_cast<const __nv_bfloat16*>(gate);
  p.ld_gate = ld_gate;
  p.out_scale = out_scale;
  p.parts = parts;
  return score_bias ? dispatch_decode<true>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s)
                    : dispatch_decode<false>(k_pages, v_pages, ld_kpage, ld_vpage, num_pages, p, s);
}

EDL_HOST_API int edl_attn_decode(const void* q, const void* k_pages, const void* v_pages, void* o, float* lse,
                                 long long ldq, long long ld_kpage, long long ld_vpage, long long ldo, const int* kv_lens,
                                 const int* page_table, int pt_stride, int B, long long num_pages, int Hq, int Hkv,
                                 int D, int Dv, float scale, int window, int keep_first, int splits, float softcap,
                                 const float* sinks, int* status, void* stream) {
  return decode_impl(q, k_pages, v_pages, o, lse, ldq, ld_kpage, ld_vpage, ldo, kv_lens, page_table, pt_stride, B, num_pages,
                     Hq, Hkv, D, Dv, scale, window, keep_first, splits, softcap, sinks, nullptr, nullptr, 0, 1.f, nullptr,
                     status, stream);
}

// The same without a softmax: a visible key's weight is sigmoid(score + score_bias[head]); the output o [B, ldo] is multiplied by
// out_scale and, with a gate [B, ld_gate] (bf16), by sigmoid(gate[b][head]). parts: workspace fp32 [splits, B, Hq * Dv] when
// splits > 1 (the parts of a plain sum need no log-sum-exp).
EDL_HOST_API int edl_attn_decode_sigmoid(const void* q, const void* k_pages, const void* v_pages, void* o, float* parts,
                                         long long ldq, long long ld_kpage, long long ld_vpage, long long ldo,
                                         const int* kv_lens, const int* page_table, int pt_stride, int B,
                                         long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int window,
                                         int keep_first, int splits, const float* score_bias, const void* gate,
                                         long long ld_gate, float out_scale, int* status, void* stream) {
  if (!score_bias || (splits > 1 && !parts)) {
    edl::set_last_error("edl_attn_decode_sigmoid: needs a bias per head, and a workspace for key splits");
    return -1;
  }
  return decode_impl(q, k_pages, v_pages, o, nullptr, ldq, ld_kpage, ld_vpage, ldo, kv_lens, page_table, pt_stride, B,
                     num_pages, Hq, Hkv, D, Dv, scale, window, keep_first, splits, 0.f, nullptr, score_bias, gate, ld_gate,
                     out_scale, parts, status, stream);
}
