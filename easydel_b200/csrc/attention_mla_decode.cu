// Decode attention over pages of latent rows (multi-head latent attention, absorbed form).
//
// The cache holds one row [compressed key/value (L) | rotary key (R)] per token, shared by every head. With the key
// up-projection folded into the query and the value up-projection applied afterwards, a decode step is
//     s[h, t] = scale * q[h, :L+R] . row[t, :L+R],   o[h, :L] = softmax_t(s[h, :]) . row[t, :L]
// i.e. an (L+R)-wide score product and an L-wide value sum over the SAME rows: every page byte is read once per group
// of 16 heads. A sliding window starts the walk at its first tile; a learned sink joins the denominator once. One CTA
// serves one (sequence, 16-head group, key split):
//   * thread 0 streams 32-row tiles (NB 64-column boxes, 128-byte swizzle, zeros past the row's end) through a
//     four-stage ring by TMA, two tiles ahead of the consumers;
//   * warp w computes the scores of rows 8w..8w+7 of the tile (4 NB m16n8k16 bf16 products against query fragments that
//     stay in registers), the four warps agree on the tile's row maxima through shared memory, write their
//     probabilities there, and each warp accumulates its own quarter of the output columns from the whole tile, so
//     the output needs no merge across warps;
//   * with key splits the partial outputs and log-sum-exps are merged by edl_attn_combine.
// L and R are multiples of 8 with L + R <= 64 NB and L <= 512.
//
// Role of the reference's multi-latent ragged page attention for decode steps
// (easydel/operations/kernels/multi_latent_ragged_page_attention.py:282-700).
#include "common.cuh"

namespace edl {
namespace {

constexpr int ML_TK = 32;              // rows per tile
constexpr int ML_WARPS = 4;
constexpr int ML_THREADS = ML_WARPS * 32;
constexpr int ML_STAGES = 4;
constexpr int ML_AHEAD = ML_STAGES - 2;
constexpr int ML_PAGE = 128;
constexpr int ML_PPITCH = ML_TK * 2 + 16;   // one row of probabilities (32 bf16) padded against bank conflicts
constexpr float ML_LOG2E = 1.4426950408889634f;

template <int NB>
struct MlCfg {
  static constexpr int W = NB * 64;                      // row width as loaded
  static constexpr int NKS = W / 16;                     // k-steps of the score product
  static constexpr int NJ = 2 * (NB < 8 ? NB : 8);       // 8-column output blocks per warp
  static constexpr int TILE_BYTES = ML_TK * W * 2;
  static constexpr int QPITCH = W * 2 + 16;
  static constexpr int OFF_Q = ML_STAGES * TILE_BYTES;
  static constexpr int OFF_P = OFF_Q + 16 * QPITCH;                // [2][16 rows][ML_PPITCH]
  static constexpr int OFF_MAX = OFF_P + 2 * 16 * ML_PPITCH;       // [2][4 warps][16] floats
  static constexpr int OFF_SUM = OFF_MAX + 2 * ML_WARPS * 16 * 4;  // [4 warps][16] floats
  static constexpr int OFF_BAR = OFF_SUM + ML_WARPS * 16 * 4;
  static constexpr int SMEM = OFF_BAR + 64 + 1024;
};

struct MlaParams {
  const __nv_bfloat16* q;   // latent part of the query: sequence b, head h at b * q_seq + h * q_head
  long long q_seq, q_head;
  const __nv_bfloat16* qr;  // rotary part, likewise
  long long qr_seq, qr_head;
  __nv_bfloat16* o;         // [splits, B, ldo]: head h at columns h * L
  long long ldo;
  float* lse;               // [splits, H, B] or null
  const int* kv_lens;
  const int* page_table;
  const float* sinks;       // [H] or null (only without splits)
  int pt_stride, B, H, splits, L, R, window;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void ml_ldmatrix_x4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ml_ldmatrix_x4_trans(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ml_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
      "{%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Byte offset of (row, 16-byte chunk) in a tile stored as nine boxes of [32 rows x 128 bytes], 128-byte swizzle.
__device__ __forceinline__ uint32_t ml_tile_off(int row, int chunk) {
  const int box = chunk >> 3, c = chunk & 7;
  return box * (ML_TK * 128) + row * 128 + ((c ^ (row & 7)) << 4);
}

template <int NB>
__global__ void __launch_bounds__(ML_THREADS, NB > 4 ? 1 : 2)
mla_decode_kernel(const __grid_constant__ CUtensorMap tmap, const MlaParams p) {
  using C = MlCfg<NB>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const uint32_t sbase = smem_u32(smem);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int groups = (p.H + 15) / 16;
  const int split = blockIdx.x % p.splits;
  const int hg = (blockIdx.x / p.splits) % groups;
  const int b = blockIdx.x / (p.splits * groups);
  const int heads = min(16, p.H - hg * 16);
  const int kv_len = p.kv_lens[b];
  const int* pt = p.page_table + (long long)b * p.pt_stride;

  const int lo = p.window > 0 ? max(0, kv_len - p.window) : 0;
  const int t_first = lo / ML_TK, t_end = (kv_len + ML_TK - 1) / ML_TK;
  const int per_split = (t_end - t_first + p.splits - 1) / p.splits;
  const int t0 = t_first + split * per_split;
  const int n_tiles = max(0, min(t_end, t0 + per_split) - t0);

  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::OFF_BAR);
  const uint32_t bar0 = smem_u32(bars);
  __shared__ int s_abort;
  if (threadIdx.x == 0) {
    for (int i = 0; i < ML_STAGES; ++i) mbar_init(bar0 + 8 * i, 1);
    s_abort = 0;
    fence_mbar_init();
    prefetch_tmap(&tmap);
  }
  {  // this group's query rows -> shared memory (rows past the last head and columns past L + R are zero)
    const __nv_bfloat16* ql = p.q + b * p.q_seq + (long long)hg * 16 * p.q_head;
    const __nv_bfloat16* qr = p.qr + b * p.qr_seq + (long long)hg * 16 * p.qr_head;
    for (int i = threadIdx.x; i < 16 * (C::W / 8); i += ML_THREADS) {
      const int r = i / (C::W / 8), c = (i % (C::W / 8)) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (r < heads && c < p.L) v = *reinterpret_cast<const uint4*>(ql + r * p.q_head + c);
      else if (r < heads && c < p.L + p.R) v = *reinterpret_cast<const uint4*>(qr + r * p.qr_head + c - p.L);
      *reinterpret_cast<uint4*>(smem + C::OFF_Q + r * C::QPITCH + c * 2) = v;
    }
  }
  __syncthreads();
  volatile int* abort_flag = &s_abort;

  auto issue = [&](int i) {  // thread 0 only
    const int tile = t0 + i;
    const int page = pt[tile / (ML_PAGE / ML_TK)];
    const int row = page * ML_PAGE + (tile % (ML_PAGE / ML_TK)) * ML_TK;
    const int st = i % ML_STAGES;
    const uint32_t bar = bar0 + 8 * st;
    const uint32_t dst = sbase + st * C::TILE_BYTES;
    mbar_expect_tx(bar, C::TILE_BYTES);
#pragma unroll
    for (int c = 0; c < NB; ++c) tma_load_2d(dst + c * (ML_TK * 128), &tmap, bar, c * 64, row);
  };
  if (threadIdx.x == 0)
    for (int i = 0; i < min(n_tiles, ML_AHEAD); ++i) issue(i);

  // A fragments of the 16 query rows for all 36 k-steps, kept in registers
  uint32_t qa[C::NKS][4];
  {
    const uint32_t qb = sbase + C::OFF_Q;
    const int r = (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int ks = 0; ks < C::NKS; ++ks) ml_ldmatrix_x4(qb + r * C::QPITCH + (ks * 2 + (lane >> 4)) * 16, qa[ks]);
  }

  float o_acc[C::NJ][4];  // this warp's quarter of the output columns: blocks of 8
#pragma unroll
  for (int j = 0; j < C::NJ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o_acc[j][e] = 0.f;
  float m_run[2] = {-1e30f, -1e30f};  // rows lane / 4 and lane / 4 + 8 (identical in every warp)
  float l_run[2] = {0.f, 0.f};        // this warp's share of the row sums (its 8 rows of every tile)
  float* s_max = reinterpret_cast<float*>(smem + C::OFF_MAX);
  bool alive = true;
  const int r0 = lane >> 2;

  for (int i = 0; i < n_tiles; ++i) {
    const int st = i % ML_STAGES, par = i & 1;
    // the stage refilled here held tile i - 2, which every warp finished before the first barrier of step i - 1
    if (threadIdx.x == 0 && i + ML_AHEAD < n_tiles && alive) issue(i + ML_AHEAD);
    if (alive) alive = mbar_wait(bar0 + 8 * st, (i / ML_STAGES) & 1, abort_flag, p.status, EDL_TIMEOUT_SOFTMAX);
    const uint32_t tile = sbase + st * C::TILE_BYTES;
    // ---- scores of rows 8w .. 8w+7 of the tile
    float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    if (alive) {                      // three independent chains of products
      const int row = warp * 8 + (lane & 7);
#pragma unroll
      for (int ks = 0; ks < C::NKS; ks += 2) {
        uint32_t kb[4];
        ml_ldmatrix_x4(tile + ml_tile_off(row, ks * 2 + (lane >> 3)), kb);
        const int chain = (ks >> 1) % 3;
        if (chain == 0) {
          ml_mma(s, qa[ks], kb[0], kb[1]);
          ml_mma(s2[0], qa[ks + 1], kb[2], kb[3]);
        } else if (chain == 1) {
          ml_mma(s2[1], qa[ks], kb[0], kb[1]);
          ml_mma(s, qa[ks + 1], kb[2], kb[3]);
        } else {
          ml_mma(s2[0], qa[ks], kb[0], kb[1]);
          ml_mma(s2[1], qa[ks + 1], kb[2], kb[3]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) s[e] += s2[0][e] + s2[1][e];
    }
    const int key0 = (t0 + i) * ML_TK + warp * 8 + (lane & 3) * 2;
    float mx[2];
#pragma unroll
    for (int e = 0; e < 4; ++e) s[e] = (alive && key0 + (e & 1) < kv_len && key0 + (e & 1) >= lo) ? s[e] * p.scale_log2 : -INFINITY;
    mx[0] = fmaxf(s[0], s[1]);
    mx[1] = fmaxf(s[2], s[3]);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
      mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
    }
    if ((lane & 3) == 0) {
      s_max[(par * ML_WARPS + warp) * 16 + r0] = mx[0];
      s_max[(par * ML_WARPS + warp) * 16 + r0 + 8] = mx[1];
    }
    __syncthreads();
    float alpha[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float m_new = m_run[h];
#pragma unroll
      for (int w = 0; w < ML_WARPS; ++w) m_new = fmaxf(m_new, s_max[(par * ML_WARPS + w) * 16 + r0 + h * 8]);
      alpha[h] = exp2f(m_run[h] - m_new);
      m_run[h] = m_new;
      l_run[h] *= alpha[h];
    }
    {  // probabilities of this warp's 8 rows -> columns 8w .. 8w+7 of the shared [16 x 32] block
      const float e0 = exp2f(s[0] - m_run[0]), e1 = exp2f(s[1] - m_run[0]);
      const float e2 = exp2f(s[2] - m_run[1]), e3 = exp2f(s[3] - m_run[1]);
      l_run[0] += e0 + e1;
      l_run[1] += e2 + e3;
      uint8_t* pb = smem + C::OFF_P + par * 16 * ML_PPITCH + (warp * 8 + (lane & 3) * 2) * 2;
      *reinterpret_cast<uint32_t*>(pb + r0 * ML_PPITCH) = pack_bf16x2(e0, e1);
      *reinterpret_cast<uint32_t*>(pb + (r0 + 8) * ML_PPITCH) = pack_bf16x2(e2, e3);
    }
    __syncthreads();
    // ---- O[:, this warp's columns] = O * alpha + P V
#pragma unroll
    for (int j = 0; j < C::NJ; ++j) {
      o_acc[j][0] *= alpha[0];
      o_acc[j][1] *= alpha[0];
      o_acc[j][2] *= alpha[1];
      o_acc[j][3] *= alpha[1];
    }
    if (alive) {
      const uint32_t pbase = sbase + C::OFF_P + par * 16 * ML_PPITCH;
#pragma unroll
      for (int t = 0; t < ML_TK / 16; ++t) {
        uint32_t pa[4];
        ml_ldmatrix_x4(pbase + ((lane & 7) + ((lane >> 3) & 1) * 8) * ML_PPITCH + (t * 2 + (lane >> 4)) * 16, pa);
#pragma unroll
        for (int j = 0; j < C::NJ; j += 2) {
          uint32_t vb[4];
          const int row = t * 16 + (lane & 7) + ((lane >> 3) & 1) * 8;
          ml_ldmatrix_x4_trans(tile + ml_tile_off(row, warp * C::NJ + j + (lane >> 4)), vb);
          ml_mma(o_acc[j], pa, vb[0], vb[1]);
          ml_mma(o_acc[j + 1], pa, vb[2], vb[3]);
        }
      }
    }
  }

  // ---- row sums over the four warps, then every warp writes its columns
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 1);
    l_run[h] += __shfl_xor_sync(0xffffffffu, l_run[h], 2);
  }
  float* s_sum = reinterpret_cast<float*>(smem + C::OFF_SUM);
  if ((lane & 3) == 0) {
    s_sum[warp * 16 + r0] = l_run[0];
    s_sum[warp * 16 + r0 + 8] = l_run[1];
  }
  __syncthreads();
  const long long orow = (long long)split * p.B + b;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int r = r0 + h * 8;
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < ML_WARPS; ++w) l += s_sum[w * 16 + r];
    if (r >= heads) continue;
    if (p.sinks && p.splits == 1) l += exp2f(p.sinks[hg * 16 + r] * ML_LOG2E - m_run[h]);
    const float inv = l > 0.f ? 1.f / l : 0.f;
    __nv_bfloat16* dst = p.o + orow * p.ldo + (long long)(hg * 16 + r) * p.L;
#pragma unroll
    for (int j = 0; j < C::NJ; ++j) {
      const int c = (warp * C::NJ + j) * 8;
      if (c < p.L) *reinterpret_cast<uint32_t*>(dst + c + (lane & 3) * 2) = pack_bf16x2(o_acc[j][2 * h] * inv, o_acc[j][2 * h + 1] * inv);
    }
    if (p.lse && warp == 0 && (lane & 3) == 0)
      p.lse[((long long)split * p.H + hg * 16 + r) * p.B + b] =
          l > 0.f ? (m_run[h] + log2f(l)) * 0.6931471805599453f : -INFINITY;
  }
  if (s_abort) {   // a wait ran out: give copies still in flight time to land before shared memory is released
    long long t0c = clock64();
    while (clock64() - t0c < 400000) {
    }
  }
}

template <int NB>
int launch_mla(const void* pages, long long num_pages, const MlaParams& p, cudaStream_t stream) {
  using C = MlCfg<NB>;
  const int w = p.L + p.R;
  CUtensorMap tm;
  if (make_tmap_2d_16b(&tm, pages, (uint64_t)num_pages * ML_PAGE, w, w, ML_TK, 64)) return -1;
  auto kern = mla_decode_kernel<NB>;
  static bool attr_set[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (dev < 0 || dev >= 64) dev = 0;
  if (!attr_set[dev]) {
    if (check_cuda(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM),
                   "cudaFuncSetAttribute(mla_decode)"))
      return -1;
    attr_set[dev] = true;
  }
  const long long blocks = (long long)p.B * ((p.H + 15) / 16) * p.splits;
  kern<<<(unsigned)blocks, ML_THREADS, C::SMEM, stream>>>(tm, p);
  return check_cuda(cudaGetLastError(), "mla_decode launch");
}

}  // namespace
}  // namespace edl

using namespace edl;

// q: latent part (L) of the absorbed queries, head h of sequence b at b * q_seq + h * q_head; qr: their rotated rotary
// part (R), likewise. pages: [num_pages, 128, L + R] bf16 rows (compressed key/value | rotated rotary key).
// o: [splits, B, ldo] bf16, head h at columns [h * L, (h + 1) * L): softmax-weighted sums of the rows' first L columns;
// lse: [splits, H, B] fp32 natural log-sum-exp without the sinks (required when splits > 1, may be null otherwise).
// kv_lens [B], page_table [B, pt_stride] int32; window: 0 or the number of latest keys a query sees (itself included);
// sinks [H] fp32 or null: an extra logit in every denominator (applied here with one split, by edl_attn_combine with
// more). scale multiplies the (L + R)-wide dot products.
EDL_HOST_API int edl_attn_mla_decode(const void* q, long long q_seq, long long q_head, const void* qr, long long qr_seq,
                                     long long qr_head, const void* pages, void* o, float* lse, long long ldo,
                                     const int* kv_lens, const int* page_table, int pt_stride, int B,
                                     long long num_pages, int H, int L, int R, float scale, int window,
                                     const float* sinks, int splits, int* status, void* stream) {
  if (B <= 0 || H <= 0) return 0;
  if (L < 8 || L > 512 || R < 0 || L + R > 576 || (L & 7) || (R & 7)) {
    set_last_error("edl_attn_mla_decode: rows of multiples of 8, latent up to 512 and 576 in all (L=%d, R=%d)", L, R);
    return -1;
  }
  if (splits < 1 || (splits > 1 && !lse) || ((q_seq | q_head | qr_seq | qr_head) & 7) || (ldo & 1) ||
      ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(qr)) & 15) || (reinterpret_cast<uintptr_t>(o) & 3)) {
    set_last_error("edl_attn_mla_decode: splits=%d needs lse; query pitches must be multiples of 8, 16-byte aligned",
                   splits);
    return -1;
  }
  MlaParams p{reinterpret_cast<const __nv_bfloat16*>(q), q_seq, q_head, reinterpret_cast<const __nv_bfloat16*>(qr), qr_seq,
              qr_head, reinterpret_cast<__nv_bfloat16*>(o), ldo, lse, kv_lens, page_table, sinks, pt_stride, B, H, splits,
              L, R, window, scale * ML_LOG2E, status};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  switch ((L + R + 63) / 64) {
    case 1: return launch_mla<1>(pages, num_pages, p, s);
    case 2: return launch_mla<2>(pages, num_pages, p, s);
    case 3: return launch_mla<3>(pages, num_pages, p, s);
    case 4: return launch_mla<4>(pages, num_pages, p, s);
    case 5: return launch_mla<5>(pages, num_pages, p, s);
    case 6: return launch_mla<6>(pages, num_pages, p, s);
    case 7: return launch_mla<7>(pages, num_pages, p, s);
    case 8: return launch_mla<8>(pages, num_pages, p, s);
    default: return launch_mla<9>(pages, num_pages, p, s);
  }
}
