// HGRN2, a gated linear recurrence without keys: a channel's write strength is the complement of its forget gate. Per
// head, with a [D, V] state S in fp32,
//
//   f_t = lower + (1 - lower) * sigmoid(z_t + bias)          (one gate per head and channel)
//   S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,   o_t = S_t^T silu(q_t)
//
// The kernels read the packed projection rows [q (H D) | z (H D) | v (H V)] and keep everything between them and the
// output in 32 bits. States live in a pool addressed by slot and are updated where they lie.
//
//   * hgrn2_decode: one token per sequence. A CTA per (sequence, head) streams the state once (it is all the traffic
//     there is), and finishes the row with the per-head RMS norm.
//   * hgrn2_scan: any number of tokens per sequence. An element-wise pass turns the projection rows into fp32 rows
//     [f (D) | silu q (D) | v (V)] per token and head. The columns of a state never meet, so a CTA owns (sequence, head,
//     column tile) and walks the tokens with its part of the state in registers: 8 rows x 4 columns per thread, packed
//     fp32 arithmetic, the rows of up to 16 tokens at a time brought into shared memory one stage ahead (cp.async).
//   * When (sequences x heads x tiles) cannot fill the GPU and sequences are long, the token axis is cut into segments:
//     one pass leaves every segment's end state from a zero start and the product of its gates, a small kernel chains
//     them into the state each segment starts from, and the scan then runs all segments at once.
//
// Compiled without fast-math.
#include "common.cuh"

namespace edl {
namespace {

__device__ __forceinline__ float g_of(float v) { return v; }
__device__ __forceinline__ float g_of(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void g_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void g_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// sigmoid in fp32. With bf16 projections the hardware exponential and divide (about 2 ulp each, far below the step of
// their operand) keep the gates off the critical path; fp32 projections take the accurate functions.
template <typename TI>
__device__ __forceinline__ float sigm(float z) {
  if constexpr (sizeof(TI) == 4) return 1.f / (1.f + expf(-z));
  else return __fdividef(1.f, 1.f + __expf(-fmaxf(z, -80.f)));
}
template <typename TI>
__device__ __forceinline__ float gate_f(float z, float lower) { return fmaf(1.f - lower, sigm<TI>(z), lower); }
template <typename TI>
__device__ __forceinline__ float silu_p(float x) { return x * sigm<TI>(x); }

// four consecutive elements of a row (vec: 4-element aligned), `n` of them real, zeros behind
template <typename TI>
__device__ __forceinline__ void load4(const TI* p, int n, bool vec, float (&v)[4]) {
  if (vec && n >= 4) {
    if constexpr (sizeof(TI) == 4) {
      const float4 a = *reinterpret_cast<const float4*>(p);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
      const uint2 a = *reinterpret_cast<const uint2*>(p);
      const float2 lo = unpack_bf16x2(a.x), hi = unpack_bf16x2(a.y);
      v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
    }
    return;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) v[j] = j < n ? g_of(p[j]) : 0.f;
}

struct Hgrn2Params {
  const void* proj;          // [T, ld]: q | z | v
  long long ld;
  const float* bias;         // [H * D]
  const float* lower;        // [H * D]
  const int* cu;             // [B + 1]
  const int* slots;          // [B] pool rows, or null: row b of the pool is sequence b
  float* state;              // pool [*, H, D, V], or null: start from zero, keep nothing
  void* out;                 // scan: fp32 [T, H * V]; decode: operand type
  int B, H, D, V;
  // segmented form
  float* ws;                 // [B * nseg, H, D, V]: end states, then start states, of the segments
  float* prod;               // [B * nseg, H, D]: products of the gates
  int seg_len, nseg;
  float* rows;               // scan: [T, H, 2 D + V] fp32 rows f | silu q | v
  int T;
  bool vec;                  // heads and rows start on 4-element boundaries
  // decode
  const float* norm;         // [V]
  float eps;
};

enum { SCAN_WHOLE = 0, SCAN_ENDS = 1, SCAN_SEGMENTS = 2 };
constexpr int SCT = 128;     // threads of a scan CTA
constexpr int CPT = 4;       // columns per thread

__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Projection rows -> fp32 rows. A thread keeps its (head, channel) and walks the tokens.
template <typename TI, int VEC>
__global__ void __launch_bounds__(256)
hgrn2_rows_kernel(const Hgrn2Params p) {
  const int D = p.D, V = p.V, width = 2 * D + V;
  const int u = blockIdx.x * 256 + threadIdx.x;
  if (u >= p.H * (width / VEC)) return;
  const int h = u / (width / VEC), c = (u - h * (width / VEC)) * VEC;
  const int kind = c < D ? 0 : (c < 2 * D ? 1 : 2);        // gate, query, value
  const int ch = h * D + (kind == 0 ? c : c - D);
  const int HD = p.H * D;
  const TI* src = reinterpret_cast<const TI*>(p.proj) +
                  (kind == 0 ? HD + ch : kind == 1 ? ch : 2 * HD + h * V + c - 2 * D);
  float b[VEC], low[VEC];
#pragma unroll
  for (int j = 0; j < VEC; ++j) {
    b[j] = kind == 0 ? p.bias[ch + j] : 0.f;
    low[j] = kind == 0 ? p.lower[ch + j] : 0.f;
  }
  float* dst = p.rows + (long long)h * width + c;
  const long long pitch = (long long)p.H * width;
#pragma unroll 4
  for (int t = blockIdx.y; t < p.T; t += gridDim.y) {
    float v[VEC];
    if constexpr (VEC == 4) load4(src + t * p.ld, 4, true, v);
    else v[0] = g_of(src[t * p.ld]);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      if (kind == 0) v[j] = gate_f<TI>(v[j] + b[j], low[j]);
      else if (kind == 1) v[j] = silu_p<TI>(v[j]);
    }
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(dst + t * pitch) = make_float4(v[0], v[1], v[2], v[3]);
    else dst[t * pitch] = v[0];
  }
}

// DP: D rounded up to a tile; RPT rows per thread; DP / RPT lanes share a column group.
template <int DP, int RPT, int MODE>
__global__ void __launch_bounds__(SCT, RPT == 8 ? 6 : 3)
hgrn2_scan_kernel(const Hgrn2Params p) {
  constexpr int SPLIT = DP / RPT;               // 4 .. 32 adjacent lanes
  constexpr int CT = (SCT / SPLIT) * CPT;       // columns of this CTA
  constexpr int TC = DP <= 128 ? 16 : 2048 / DP;   // tokens per stage
  constexpr int NK = RPT / 4;
  constexpr bool Q = MODE != SCAN_ENDS;
  static_assert(SPLIT >= 4 && SPLIT <= 32 && RPT % 4 == 0, "");
  __shared__ __align__(16) float sf[2][TC][DP];
  __shared__ __align__(16) float sq[2][Q ? TC : 1][DP];
  __shared__ __align__(16) float sv[2][TC][CT];
  const int tid = threadIdx.x;
  const int part = tid % SPLIT, grp = tid / SPLIT;
  const int h = blockIdx.y;
  const int col0 = blockIdx.x * CT, col = col0 + grp * CPT;
  int b, seg = 0, t0, t1;
  if (MODE == SCAN_WHOLE) {
    b = blockIdx.z;
    t0 = p.cu[b];
    t1 = p.cu[b + 1];
  } else {
    b = blockIdx.z / p.nseg;
    seg = blockIdx.z % p.nseg;
    t0 = p.cu[b] + seg * p.seg_len;
    t1 = min(p.cu[b + 1], t0 + p.seg_len);
  }
  if (t0 >= t1) return;
  const bool final_seg = MODE == SCAN_WHOLE || t1 == p.cu[b + 1];
  if (MODE == SCAN_ENDS && final_seg) return;   // nothing follows the last segment
  const long long mat = (long long)p.D * p.V;
  float* pool = nullptr;
  if (p.state) pool = p.state + ((long long)(p.slots ? p.slots[b] : b) * p.H + h) * mat;
  float* seg_state = MODE == SCAN_WHOLE ? nullptr : p.ws + ((long long)(b * p.nseg + seg) * p.H + h) * mat;

  // the stages' columns past the real sizes are zeros: the copies never touch them
  if (p.D < DP) {
    for (int i = tid; i < 2 * TC * DP; i += SCT) {
      (&sf[0][0][0])[i] = 0.f;
      if (Q) (&sq[0][0][0])[i] = 0.f;
    }
  }
  if (col0 + CT > p.V)
    for (int i = tid; i < 2 * TC * CT; i += SCT) (&sv[0][0][0])[i] = 0.f;
  __syncthreads();
  const int width = 2 * p.D + p.V;
  auto fetch = [&](int tb, int buf) {
    const int n = min(TC, t1 - tb);
    const float* base = p.rows + ((long long)tb * p.H + h) * width;
    const long long pitch = (long long)p.H * width;
    for (int i = tid; i < n * (DP / 4); i += SCT) {
      const int t = i / (DP / 4), d = (i % (DP / 4)) * 4;
      const float* row = base + t * pitch + d;
      if (p.vec) {
        if (d < p.D) {
          cp_async16(&sf[buf][t][d], row);
          if (Q) cp_async16(&sq[buf][t][d], row + p.D);
        }
      } else {
        for (int j = 0; j < 4 && d + j < p.D; ++j) {
          sf[buf][t][d + j] = row[j];
          if (Q) sq[buf][t][d + j] = row[p.D + j];
        }
      }
    }
    for (int i = tid; i < n * (CT / 4); i += SCT) {
      const int t = i / (CT / 4), c = (i % (CT / 4)) * 4;
      const float* row = base + t * pitch + 2 * p.D + col0 + c;
      if (p.vec) {
        if (col0 + c < p.V) cp_async16(&sv[buf][t][c], row);
      } else {
        for (int j = 0; j < 4 && col0 + c + j < p.V; ++j) sv[buf][t][c + j] = row[j];
      }
    }
    cp_async_commit();
  };
  fetch(t0, 0);

  // rows of this thread: 4 * (part + SPLIT * k) + j, k < NK, j < 4; packed arithmetic takes rows j, j + 1 as a pair
  float S[NK][4][CPT];
  float pr[NK][4];
  {
    const float* src = MODE == SCAN_WHOLE ? pool : (MODE == SCAN_SEGMENTS ? seg_state : nullptr);
#pragma unroll
    for (int k = 0; k < NK; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = 4 * (part + SPLIT * k) + j;
        pr[k][j] = 1.f;
#pragma unroll
        for (int c = 0; c < CPT; ++c)
          S[k][j][c] = (src && row < p.D && col + c < p.V) ? src[(long long)row * p.V + col + c] : 0.f;
      }
  }
  float* out = reinterpret_cast<float*>(p.out) + ((long long)t0 * p.H + h) * p.V + col + (part & 1) * 2 + ((part >> 1) & 1);
  const bool writes = part < 4 && col + (part & 1) * 2 + ((part >> 1) & 1) < p.V;
  int buf = 0;
  for (int tb = t0; tb < t1; tb += TC, buf ^= 1) {
    const int n = min(TC, t1 - tb);
    if (tb + TC < t1) {
      fetch(tb + TC, buf ^ 1);     // every warp left that stage at the barrier below
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
#pragma unroll 2
    for (int t = 0; t < n; ++t) {
      const float4 v4 = *reinterpret_cast<const float4*>(&sv[buf][t][grp * CPT]);
      const float v[CPT] = {v4.x, v4.y, v4.z, v4.w};
      float a0[CPT], a1[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) a0[c] = a1[c] = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        const float4 f4 = *reinterpret_cast<const float4*>(&sf[buf][t][4 * (part + SPLIT * k)]);
        float4 q4 = make_float4(0.f, 0.f, 0.f, 0.f);
        if (MODE != SCAN_ENDS) q4 = *reinterpret_cast<const float4*>(&sq[buf][t][4 * (part + SPLIT * k)]);
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          // S = f S + (1 - f) v as v + f (S - v), two rows per instruction
          float d0 = S[k][0][c], d1 = S[k][1][c], d2 = S[k][2][c], d3 = S[k][3][c];
          add2(d0, d1, -v[c], -v[c]);
          add2(d2, d3, -v[c], -v[c]);
          fma2(S[k][0][c], S[k][1][c], f4.x, f4.y, d0, d1, v[c], v[c]);
          fma2(S[k][2][c], S[k][3][c], f4.z, f4.w, d2, d3, v[c], v[c]);
          if (MODE != SCAN_ENDS) {
            fma2(a0[c], a1[c], q4.x, q4.y, S[k][0][c], S[k][1][c], a0[c], a1[c]);
            fma2(a0[c], a1[c], q4.z, q4.w, S[k][2][c], S[k][3][c], a0[c], a1[c]);
          }
        }
        if (MODE == SCAN_ENDS) {
          pr[k][0] *= f4.x;
          pr[k][1] *= f4.y;
          pr[k][2] *= f4.z;
          pr[k][3] *= f4.w;
        }
      }
      if (MODE != SCAN_ENDS) {
        // sum over the lanes of the group: the first two exchanges also spread the four columns over four lanes
        float s[CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) s[c] = a0[c] + a1[c];
        const bool hi0 = part & 1, hi1 = part & 2;
        const float x0 = __shfl_xor_sync(0xffffffffu, hi0 ? s[0] : s[2], 1);
        const float x1 = __shfl_xor_sync(0xffffffffu, hi0 ? s[1] : s[3], 1);
        const float y0 = (hi0 ? s[2] : s[0]) + x0, y1 = (hi0 ? s[3] : s[1]) + x1;
        float z = (hi1 ? y1 : y0) + __shfl_xor_sync(0xffffffffu, hi1 ? y0 : y1, 2);
#pragma unroll
        for (int o = 4; o < SPLIT; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        if (writes) *out = z;
        out += (long long)p.H * p.V;
      }
    }
    __syncthreads();
  }
  float* dst = MODE == SCAN_ENDS ? seg_state : (final_seg ? pool : nullptr);
  if (dst) {
#pragma unroll
    for (int k = 0; k < NK; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = 4 * (part + SPLIT * k) + j;
        if (row < p.D) {
#pragma unroll
          for (int c = 0; c < CPT; ++c)
            if (col + c < p.V) dst[(long long)row * p.V + col + c] = S[k][j][c];
          if (MODE == SCAN_ENDS && col == 0)
            p.prod[((long long)(b * p.nseg + seg) * p.H + h) * p.D + row] = pr[k][j];
        }
      }
  }
}

// Start state of every segment from the pool state, the end states and the gate products.
__global__ void hgrn2_chain_kernel(const Hgrn2Params p) {
  const int b = blockIdx.z, h = blockIdx.y;
  const int len = p.cu[b + 1] - p.cu[b];
  if (len <= 0) return;
  const int segs = (len + p.seg_len - 1) / p.seg_len;
  const long long mat = (long long)p.D * p.V;
  const float* pool = p.state ? p.state + ((long long)(p.slots ? p.slots[b] : b) * p.H + h) * mat : nullptr;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < mat;
       i += (long long)gridDim.x * blockDim.x) {
    const int row = (int)(i / p.V);
    float s = pool ? pool[i] : 0.f;
    constexpr int AHEAD = 8;                     // segments whose loads are in flight together
    for (int g0 = 0; g0 < segs; g0 += AHEAD) {
      float end[AHEAD], f[AHEAD];
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        const long long at = (long long)(b * p.nseg + g0 + j) * p.H + h;
        if (g0 + j + 1 < segs) {
          end[j] = p.ws[at * mat + i];
          f[j] = p.prod[at * p.D + row];
        }
      }
#pragma unroll
      for (int j = 0; j < AHEAD; ++j) {
        if (g0 + j >= segs) break;
        p.ws[((long long)(b * p.nseg + g0 + j) * p.H + h) * mat + i] = s;
        if (g0 + j + 1 < segs) s = fmaf(f[j], s, end[j]);
      }
    }
  }
}

constexpr int DCT = 256;

// One token per sequence; VEC columns per thread.
template <typename TI, int VEC>
__global__ void __launch_bounds__(DCT)
hgrn2_decode_kernel(const Hgrn2Params p) {
  extern __shared__ __align__(16) float dsm[];   // f [D] | q [D] | partial sums [groups][V]
  __shared__ float red[32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const TI* row = reinterpret_cast<const TI*>(p.proj) + (long long)p.cu[b] * p.ld;
  if (p.cu[b + 1] <= p.cu[b]) return;
  const int HD = p.H * p.D, D = p.D, V = p.V;
  float* sf = dsm;
  float* sq = dsm + D;
  float* sums = dsm + ((2 * D + 3) & ~3);
  const int vcols = V / VEC;                     // column groups
  const int groups = max(1, DCT / vcols);        // row groups
  float* st = p.state + ((long long)(p.slots ? p.slots[b] : b) * p.H + h) * (long long)D * V;
  for (int d = tid; d < D; d += DCT) {
    sf[d] = gate_f<TI>(g_of(row[HD + h * D + d]) + p.bias[h * D + d], p.lower[h * D + d]);
    sq[d] = silu_p<TI>(g_of(row[h * D + d]));
  }
  __syncthreads();
  for (int u = tid; u < vcols * groups; u += DCT) {   // one round unless V / VEC > DCT
    const int cg = u % vcols, rg = u / vcols;
    float v[VEC], acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      v[j] = g_of(row[2 * HD + h * V + cg * VEC + j]);
      acc[j] = 0.f;
    }
    constexpr int BATCH = 8;                     // rows in flight: all loads of a batch are issued before its stores
    for (int d0 = rg; d0 < D; d0 += groups * BATCH) {
      float s[BATCH][VEC];
#pragma unroll
      for (int i = 0; i < BATCH; ++i) {
        const int d = d0 + i * groups;
        const float* sp = st + (long long)d * V + cg * VEC;
        if (d < D) {
          if constexpr (VEC == 4) {
            const float4 x = *reinterpret_cast<const float4*>(sp);
            s[i][0] = x.x; s[i][1] = x.y; s[i][2] = x.z; s[i][3] = x.w;
          } else {
#pragma unroll
            for (int j = 0; j < VEC; ++j) s[i][j] = sp[j];
          }
        }
      }
#pragma unroll
      for (int i = 0; i < BATCH; ++i) {
        const int d = d0 + i * groups;
        if (d >= D) break;
        float* sp = st + (long long)d * V + cg * VEC;
        const float f = sf[d], q = sq[d];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          s[i][j] = fmaf(f, s[i][j] - v[j], v[j]);
          acc[j] = fmaf(q, s[i][j], acc[j]);
        }
        if constexpr (VEC == 4) {
          *reinterpret_cast<float4*>(sp) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
        } else {
#pragma unroll
          for (int j = 0; j < VEC; ++j) sp[j] = s[i][j];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) sums[rg * V + cg * VEC + j] = acc[j];
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < V; c += DCT) {
    float o = 0.f;
    for (int g = 0; g < groups; ++g) o += sums[g * V + c];
    sums[c] = o;                                 // group 0's own place
    ss += o * o;
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)V + p.eps);
  TI* out = reinterpret_cast<TI*>(p.out) + (long long)p.cu[b] * p.H * V + (long long)h * V;
  for (int c = tid; c < V; c += DCT) g_put(out + c, sums[c] * rs * p.norm[c]);
}

template <int MODE>
int launch_scan(const Hgrn2Params& p, int z, cudaStream_t s) {
#define EDL_HS(DP, RPT)                                                                          \
  {                                                                                              \
    constexpr int CT = (SCT / (DP / RPT)) * CPT;                                                 \
    hgrn2_scan_kernel<DP, RPT, MODE><<<dim3((p.V + CT - 1) / CT, p.H, z), SCT, 0, s>>>(p);   \
  }
  if (p.D <= 32) EDL_HS(32, 8)
  else if (p.D <= 64) EDL_HS(64, 8)
  else if (p.D <= 128) EDL_HS(128, 8)
  else if (p.D <= 256) EDL_HS(256, 8)
  else EDL_HS(512, 16)
#undef EDL_HS
  return check_cuda(cudaGetLastError(), "hgrn2_scan launch");
}

template <typename TI>
int run_scan(Hgrn2Params& p, cudaStream_t s) {
  const int per_token = p.H * ((2 * p.D + p.V) / (p.vec ? 4 : 1));
  const int gx = (per_token + 255) / 256;
  int gy = (8 * sm_count() + gx - 1) / gx;
  if (gy > p.T) gy = p.T;
  if (p.vec) hgrn2_rows_kernel<TI, 4><<<dim3(gx, gy), 256, 0, s>>>(p);
  else hgrn2_rows_kernel<TI, 1><<<dim3(gx, gy), 256, 0, s>>>(p);
  if (check_cuda(cudaGetLastError(), "hgrn2_rows launch")) return -1;
  if (p.seg_len <= 0) return launch_scan<SCAN_WHOLE>(p, p.B, s);
  if (launch_scan<SCAN_ENDS>(p, p.B * p.nseg, s)) return -1;
  const long long mat = (long long)p.D * p.V;
  hgrn2_chain_kernel<<<dim3((unsigned)((mat + 255) / 256), p.H, p.B), 256, 0, s>>>(p);
  if (check_cuda(cudaGetLastError(), "hgrn2_chain launch")) return -1;
  return launch_scan<SCAN_SEGMENTS>(p, p.B * p.nseg, s);
}

bool bad_sizes(const char* who, int B, int H, int D, int V) {
  if (H < 1 || H > 65535 || D < 1 || D > 512 || V < 1 || V > 1024 || B > 65535) {
    set_last_error("%s: unsupported sizes (B=%d, H=%d, D=%d, V=%d)", who, B, H, D, V);
    return true;
  }
  return false;
}

}  // namespace
}  // namespace edl

using namespace edl;

// o [T, H * V] fp32 (no output norm); rows: workspace [T, H, 2 D + V] fp32. seg_len > 0: segmented form, nseg >= ceil(longest sequence / seg_len), with
// ws [B * nseg, H, D, V] and prod [B * nseg, H, D] fp32.
EDL_HOST_API int edl_hgrn2_scan(const void* proj, int f32, long long ld, const float* bias, const float* lower,
                                const int* cu, const int* slots, float* state, float* o, float* rows, int T, int B,
                                int H, int D, int V, int seg_len, int nseg, float* ws, float* prod, void* stream) {
  if (B <= 0 || T <= 0) return 0;
  if (bad_sizes("edl_hgrn2_scan", B, H, D, V)) return -1;
  if (seg_len > 0 && (nseg < 1 || !ws || !prod || (long long)B * nseg > 65535)) {
    set_last_error("edl_hgrn2_scan: bad segmentation (seg_len=%d, nseg=%d)", seg_len, nseg);
    return -1;
  }
  Hgrn2Params p{};
  p.proj = proj; p.ld = ld; p.bias = bias; p.lower = lower; p.cu = cu; p.slots = slots; p.state = state; p.out = o;
  p.B = B; p.H = H; p.D = D; p.V = V; p.seg_len = seg_len; p.nseg = nseg; p.ws = ws; p.prod = prod;
  p.rows = rows; p.T = T;
  p.vec = D % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(proj) & (f32 ? 15 : 7)) == 0 &&
          (reinterpret_cast<uintptr_t>(rows) & 15) == 0;
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? run_scan<float>(p, s) : run_scan<__nv_bfloat16>(p, s);
}

// One token per sequence (row cu[b] of proj), output norm included; out [T, H * V] in the projection's type.
EDL_HOST_API int edl_hgrn2_decode(const void* proj, int f32, long long ld, const float* bias, const float* lower,
                                  const int* cu, const int* slots, float* state, const float* norm, float eps,
                                  void* out, int B, int H, int D, int V, void* stream) {
  if (B <= 0) return 0;
  if (bad_sizes("edl_hgrn2_decode", B, H, D, V)) return -1;
  if (!state) {
    set_last_error("edl_hgrn2_decode: needs a state pool");
    return -1;
  }
  Hgrn2Params p{};
  p.proj = proj; p.ld = ld; p.bias = bias; p.lower = lower; p.cu = cu; p.slots = slots; p.state = state; p.out = out;
  p.B = B; p.H = H; p.D = D; p.V = V; p.norm = norm; p.eps = eps;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = V % 4 == 0 && (reinterpret_cast<uintptr_t>(state) & 15) == 0;
  const int vcols = v4 ? V / 4 : V;
  const int groups = vcols >= DCT ? 1 : DCT / vcols;
  const size_t smem = (size_t)(((2 * D + 3) & ~3) + groups * V) * sizeof(float);   // <= 2 * 512 + 1024 + V floats
  const dim3 grid(H, B);
#define EDL_HD(T, V_) hgrn2_decode_kernel<T, V_><<<grid, DCT, smem, s>>>(p)
  if (f32) {
    if (v4) EDL_HD(float, 4); else EDL_HD(float, 1);
  } else {
    if (v4) EDL_HD(__nv_bfloat16, 4); else EDL_HD(__nv_bfloat16, 1);
  }
#undef EDL_HD
  return check_cuda(cudaGetLastError(), "hgrn2_decode launch");
}
