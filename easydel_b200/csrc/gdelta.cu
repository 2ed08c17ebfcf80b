// Generalised delta rule: a linear recurrence whose state forgets per channel and removes what it holds along one direction.
// Per head, with a [D, V] state S in fp32,
//
//   u_t = k_t / sqrt(|k_t|^2 + c),   w_t = exp(-rate * sigmoid(z_t + w0)),   a_t = sigmoid(y_t + a0)      (per key channel)
//   S_t = diag(w_t) S_{t-1} - (a_t u_t) (u_t^T S_{t-1}) + k_t v_t^T,   o_t = S_t^T r_t
//
// and each head's o leaves RMS-normed, times a weight, times sigmoid(gate). z is a product of low rank, W2 tanh(x). The
// kernels read columns of one packed projection (r, k, v, a, gate, x) and keep everything between it and the output in 32
// bits. States live in a pool addressed by slot and are updated where they lie.
//
//   * gdelta_decode: one token per sequence. A CTA per (sequence, head) holds the state in registers between the product
//     with u and the update, so it is read once and written once; it also forms z and finishes the row.
//   * gdelta_rows + gdelta_scan + gdelta_finish: any number of tokens. The rows pass leaves fp32 rows [w | u | a u | r |
//     |k| v] per token and head (k v^T = u (|k| v)^T). The columns of a state never meet, so a scan CTA owns (sequence, head,
//     column tile) and walks the tokens with its part of the state in registers, packed fp32 arithmetic, rows brought into
//     shared memory one stage ahead (cp.async).
//
// Compiled without fast-math.
#include "common.cuh"

namespace edl {
namespace {

__device__ __forceinline__ float d_of(float v) { return v; }
__device__ __forceinline__ float d_of(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void d_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void d_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

__device__ __forceinline__ float sigm(float z) { return 1.f / (1.f + expf(-z)); }

template <int VEC, typename T>
__device__ __forceinline__ void d_load(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else if constexpr (VEC == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack_bf16x2(a.x), hi = unpack_bf16x2(a.y);
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = d_of(p[i]);
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void d_store(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (VEC == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) d_put(p + i, v[i]);
  }
}

struct DeltaParams {
  const void *r, *k, *v, *a, *g, *x;   // columns of the packed projection (operand type), row pitch ld
  long long ld;
  const float* z;            // scan: [T, H * D] fp32 low-rank product
  const void* w2;            // decode: [H * D, rank] operand type
  int rank;
  const float *w0, *a0;      // [H * D]
  float rate, unit_eps;
  const int* cu;             // [B + 1]
  const int* slots;          // [B] pool rows, or null: row b of the pool is sequence b
  float* state;              // pool [*, H, D, V], or null: start from zero, keep nothing
  float* o;                  // scan: [T, H * V]
  float* rows;               // scan: [T, H, 4 D + V] w | u | a u | r | |k| v
  const float* norm;         // [H * V]
  float eps, scale;          // of the output: norm epsilon, factor
  void* out;                 // operand type, row pitch ld_out
  long long ld_out;
  int T, B, H, D, V;
  bool vec;
};

// ---- rows -----------------------------------------------------------------------------------------------------------
constexpr int RT = 256;

// LANES adjacent lanes per (token, head).
template <typename T, int VEC>
__global__ void __launch_bounds__(RT) gdelta_rows_kernel(const DeltaParams p, int lanes) {
  const int D = p.D, V = p.V, width = 4 * D + V;
  const int sub = threadIdx.x % lanes;
  const long long items = (long long)p.T * p.H, stride = (long long)gridDim.x * (RT / lanes);
  const long long rounds = (items + stride - 1) / stride;      // the same for every lane: the sums are warp-wide exchanges
  long long it = blockIdx.x * (long long)(RT / lanes) + threadIdx.x / lanes;
  for (long long n = 0; n < rounds; ++n, it += stride) {
    const bool live = it < items;
    const long long t = live ? it / p.H : 0;
    const int h = live ? (int)(it - t * p.H) : 0;
    const T* k = reinterpret_cast<const T*>(p.k) + t * p.ld + (long long)h * D;
    float ss = 0.f;
    if (live)
      for (int c = sub * VEC; c < D; c += lanes * VEC) {
        float b[VEC];
        d_load<VEC>(k + c, b);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += b[j] * b[j];
      }
    for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live) continue;
    const float len = sqrtf(ss + p.unit_eps), inv = 1.f / len;
    float* dst = p.rows + it * width;
    const T* r = reinterpret_cast<const T*>(p.r) + t * p.ld + (long long)h * D;
    const T* a = reinterpret_cast<const T*>(p.a) + t * p.ld + (long long)h * D;
    const float* z = p.z + it * D;
    for (int c = sub * VEC; c < D; c += lanes * VEC) {
      float b[VEC], zz[VEC], w0[VEC], a0[VEC], u[VEC], w[VEC], rr[VEC];
      d_load<VEC>(k + c, u);
      d_load<VEC>(a + c, b);
      d_load<VEC>(r + c, rr);
      d_load<VEC>(z + c, zz);
      d_load<VEC>(p.w0 + h * D + c, w0);
      d_load<VEC>(p.a0 + h * D + c, a0);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        u[j] *= inv;
        b[j] = sigm(b[j] + a0[j]) * u[j];
        w[j] = expf(-p.rate * sigm(zz[j] + w0[j]));
      }
      d_store<VEC>(dst + c, w);
      d_store<VEC>(dst + D + c, u);
      d_store<VEC>(dst + 2 * D + c, b);
      d_store<VEC>(dst + 3 * D + c, rr);
    }
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.ld + (long long)h * V;
    for (int c = sub * VEC; c < V; c += lanes * VEC) {
      float b[VEC];
      d_load<VEC>(v + c, b);
#pragma unroll
      for (int j = 0; j < VEC; ++j) b[j] *= len;
      d_store<VEC>(dst + 4 * D + c, b);
    }
  }
}

// ---- scan -----------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// DP: D rounded up to a tile; a thread holds RPT rows x CPT columns, DP / RPT adjacent lanes share the columns.
template <int DP, int RPT, int CPT, int NT>
struct ScanCfg {
  static constexpr int SPLIT = DP / RPT;
  static constexpr int CT = (NT / SPLIT) * CPT;                 // columns of a CTA
  static constexpr int TC = DP <= 64 ? 16 : 1024 / DP;          // tokens per stage
  static constexpr int CTP = (CT + 3) / 4 * 4;
  static constexpr int STAGE = TC * (4 * DP + CTP);             // floats
};

template <int DP, int RPT, int CPT, int NT>
__global__ void __launch_bounds__(NT, 256 / NT) gdelta_scan_kernel(const DeltaParams p) {
  using C = ScanCfg<DP, RPT, CPT, NT>;
  constexpr int SPLIT = C::SPLIT, CT = C::CT, TC = C::TC, NK = RPT / 4;
  static_assert(SPLIT >= CPT && SPLIT <= 32 && RPT % 4 == 0 && (CPT == 1 || CPT == 2 || CPT == 4), "");
  extern __shared__ __align__(16) float smem[];
  const int tid = threadIdx.x;
  const int part = tid % SPLIT, grp = tid / SPLIT;
  const int h = blockIdx.y, b = blockIdx.z;
  const int col0 = blockIdx.x * CT, col = col0 + grp * CPT;
  const int t0 = p.cu[b], t1 = p.cu[b + 1];
  if (t0 >= t1) return;
  const int D = p.D, V = p.V, width = 4 * D + V;
  float* pool = p.state ? p.state + ((long long)(p.slots ? p.slots[b] : b) * p.H + h) * (long long)D * V : nullptr;

  // the stages' columns past the real sizes are zeros: the copies never touch them
  if (D < DP || col0 + CT > V) {
    for (int i = tid; i < 2 * C::STAGE; i += NT) smem[i] = 0.f;
    __syncthreads();
  }
  // stage layout: [4][TC][DP] w | u | a u | r, then [TC][CTP] values
  auto fetch = [&](int tb, int buf) {
    float* st = smem + buf * C::STAGE;
    const int n = min(TC, t1 - tb);
    const float* base = p.rows + ((long long)tb * p.H + h) * width;
    const long long pitch = (long long)p.H * width;
    for (int i = tid; i < n * (DP / 4); i += NT) {
      const int t = i / (DP / 4), d = (i % (DP / 4)) * 4;
      const float* row = base + t * pitch + d;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float* dst = st + (q * TC + t) * DP + d;
        if (p.vec) {
          if (d < D) cp_async16(dst, row + q * D);
        } else {
          for (int j = 0; j < 4 && d + j < D; ++j) dst[j] = row[q * D + j];
        }
      }
    }
    for (int i = tid; i < n * (C::CTP / 4); i += NT) {
      const int t = i / (C::CTP / 4), c = (i % (C::CTP / 4)) * 4;
      const float* row = base + t * pitch + 4 * D + col0 + c;
      float* dst = st + 4 * TC * DP + t * C::CTP + c;
      if (p.vec) {
        if (col0 + c < V) cp_async16(dst, row);
      } else {
        for (int j = 0; j < 4 && col0 + c + j < V; ++j) dst[j] = row[j];
      }
    }
    cp_async_commit();
  };
  fetch(t0, 0);

  // rows of this thread: 4 * (part + SPLIT * i) + j, i < NK, j < 4; packed arithmetic takes rows j, j + 1 as a pair
  float S[NK][4][CPT];
#pragma unroll
  for (int i = 0; i < NK; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = 4 * (part + SPLIT * i) + j;
#pragma unroll
      for (int c = 0; c < CPT; ++c) S[i][j][c] = (pool && row < D && col + c < V) ? pool[(long long)row * V + col + c] : 0.f;
    }
  // column whose output this lane writes
  const int mine = CPT == 4 ? (part & 1) * 2 + ((part >> 1) & 1) : CPT == 2 ? (part & 1) : 0;
  const unsigned pitch = (unsigned)p.H * V;
  float* out = p.o + ((long long)t0 * p.H + h) * V + col + mine;       // where the next `late` goes: the first one is no
  const bool writes = part < CPT && col + mine < V;                    // token's and is written over
  unsigned step = 0;
  // The lanes' sums over a column are the longest wait of a token: those of the outputs are taken one token late, together
  // with the next token's u^T S, and diag(w) S + u v^T is formed while both are on their way.
  constexpr int STEPS = SPLIT == 4 ? 2 : SPLIT == 8 ? 3 : SPLIT == 16 ? 4 : 5;
  float late[CPT];
#pragma unroll
  for (int c = 0; c < CPT; ++c) late[c] = 0.f;
  // step q of the sum of the outputs; the first steps also spread the columns over lanes
  auto late_step = [&](int q) {
    if (CPT == 4 && q == 0) {
      const bool hi = part & 1;
      const float x0 = __shfl_xor_sync(0xffffffffu, hi ? late[0] : late[2 % CPT], 1);
      const float x1 = __shfl_xor_sync(0xffffffffu, hi ? late[1 % CPT] : late[3 % CPT], 1);
      late[0] = (hi ? late[2 % CPT] : late[0]) + x0;
      late[1 % CPT] = (hi ? late[3 % CPT] : late[1 % CPT]) + x1;
    } else if ((CPT == 4 && q == 1) || (CPT == 2 && q == 0)) {
      const bool hi = part & (1 << q);
      const float x = __shfl_xor_sync(0xffffffffu, hi ? late[0] : late[1 % CPT], 1 << q);
      late[0] = (hi ? late[1 % CPT] : late[0]) + x;
    } else {
      late[0] += __shfl_xor_sync(0xffffffffu, late[0], 1 << q);
    }
  };
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
    const float* st = smem + buf * C::STAGE;
    const float* sw = st + 4 * part;
    const float* sv = st + 4 * TC * DP + grp * CPT;
    float4 u4[NK];
#pragma unroll
    for (int i = 0; i < NK; ++i) u4[i] = *reinterpret_cast<const float4*>(sw + TC * DP + 4 * SPLIT * i);
#pragma unroll 2
    for (int t = 0; t < n; ++t, sw += DP, sv += C::CTP) {
      float v[CPT], d[CPT][4], seen[CPT];
      float4 w4[NK], b4[NK], r4[NK];
#pragma unroll
      for (int c = 0; c < CPT; ++c) v[c] = sv[c];
#pragma unroll
      for (int i = 0; i < NK; ++i) w4[i] = *reinterpret_cast<const float4*>(sw + 4 * SPLIT * i);
#pragma unroll
      for (int i = 0; i < NK; ++i)
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          if (i == 0) {
            mul2(d[c][0], d[c][1], u4[i].x, u4[i].y, S[i][0][c], S[i][1][c]);
            mul2(d[c][2], d[c][3], u4[i].z, u4[i].w, S[i][2][c], S[i][3][c]);
          } else {
            fma2(d[c][0], d[c][1], u4[i].x, u4[i].y, S[i][0][c], S[i][1][c], d[c][0], d[c][1]);
            fma2(d[c][2], d[c][3], u4[i].z, u4[i].w, S[i][2][c], S[i][3][c], d[c][2], d[c][3]);
          }
        }
#pragma unroll
      for (int i = 0; i < NK; ++i) {
        b4[i] = *reinterpret_cast<const float4*>(sw + 2 * TC * DP + 4 * SPLIT * i);
        r4[i] = *reinterpret_cast<const float4*>(sw + 3 * TC * DP + 4 * SPLIT * i);
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        add2(d[c][0], d[c][1], d[c][2], d[c][3]);
        seen[c] = d[c][0] + d[c][1];
      }
      // a share of diag(w) S + u v^T behind every exchange
      constexpr int SHARE = (NK + STEPS - 1) / STEPS;
#pragma unroll
      for (int q = 0; q < STEPS; ++q) {
        float more[CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) more[c] = __shfl_xor_sync(0xffffffffu, seen[c], 1 << q);
        late_step(q);
#pragma unroll
        for (int i = q * SHARE; i < (q + 1) * SHARE && i < NK; ++i)
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            float x0, x1, x2, x3;
            mul2(x0, x1, u4[i].x, u4[i].y, v[c], v[c]);
            mul2(x2, x3, u4[i].z, u4[i].w, v[c], v[c]);
            fma2(S[i][0][c], S[i][1][c], w4[i].x, w4[i].y, S[i][0][c], S[i][1][c], x0, x1);
            fma2(S[i][2][c], S[i][3][c], w4[i].z, w4[i].w, S[i][2][c], S[i][3][c], x2, x3);
          }
#pragma unroll
        for (int c = 0; c < CPT; ++c) seen[c] += more[c];
      }
      if (writes) *out = late[0];
      out += step;
      step = pitch;
      {
        const float* next = sw + (t + 1 < n ? TC + 1 : TC) * DP;
#pragma unroll
        for (int i = 0; i < NK; ++i) u4[i] = *reinterpret_cast<const float4*>(next + 4 * SPLIT * i);
      }
      float a[CPT][4];
#pragma unroll
      for (int i = 0; i < NK; ++i)
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          fma2(S[i][0][c], S[i][1][c], b4[i].x, b4[i].y, -seen[c], -seen[c], S[i][0][c], S[i][1][c]);
          fma2(S[i][2][c], S[i][3][c], b4[i].z, b4[i].w, -seen[c], -seen[c], S[i][2][c], S[i][3][c]);
          if (i == 0) {
            mul2(a[c][0], a[c][1], r4[i].x, r4[i].y, S[i][0][c], S[i][1][c]);
            mul2(a[c][2], a[c][3], r4[i].z, r4[i].w, S[i][2][c], S[i][3][c]);
          } else {
            fma2(a[c][0], a[c][1], r4[i].x, r4[i].y, S[i][0][c], S[i][1][c], a[c][0], a[c][1]);
            fma2(a[c][2], a[c][3], r4[i].z, r4[i].w, S[i][2][c], S[i][3][c], a[c][2], a[c][3]);
          }
        }
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        add2(a[c][0], a[c][1], a[c][2], a[c][3]);
        late[c] = a[c][0] + a[c][1];
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int q = 0; q < STEPS; ++q) late_step(q);        // the last token's output
  if (writes) *out = late[0];
  if (pool) {
#pragma unroll
    for (int i = 0; i < NK; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = 4 * (part + SPLIT * i) + j;
#pragma unroll
        for (int c = 0; c < CPT; ++c)
          if (row < D && col + c < V) pool[(long long)row * V + col + c] = S[i][j][c];
      }
  }
}

// ---- output norm and gate -------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(RT) gdelta_finish_kernel(const DeltaParams p, int lanes) {
  const int V = p.V, sub = threadIdx.x % lanes;
  const long long items = (long long)p.T * p.H, stride = (long long)gridDim.x * (RT / lanes);
  const long long rounds = (items + stride - 1) / stride;
  long long it = blockIdx.x * (long long)(RT / lanes) + threadIdx.x / lanes;
  for (long long n = 0; n < rounds; ++n, it += stride) {
    const bool live = it < items;
    const float* o = p.o + it * V;
    float ss = 0.f;
    if (live)
      for (int c = sub * VEC; c < V; c += lanes * VEC) {
        float b[VEC];
        d_load<VEC>(o + c, b);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += b[j] * b[j];
      }
    for (int s = lanes >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
    if (!live) continue;
    const float f = p.scale / sqrtf(ss / (float)V + p.eps);
    const long long t = it / p.H;
    const int h = (int)(it - t * p.H);
    const T* g = reinterpret_cast<const T*>(p.g) + t * p.ld + (long long)h * V;
    T* dst = reinterpret_cast<T*>(p.out) + t * p.ld_out + (long long)h * V;
    for (int c = sub * VEC; c < V; c += lanes * VEC) {
      float b[VEC], gg[VEC], w[VEC];
      d_load<VEC>(o + c, b);
      d_load<VEC>(g + c, gg);
      d_load<VEC>(p.norm + h * V + c, w);
#pragma unroll
      for (int j = 0; j < VEC; ++j) b[j] = b[j] * f * w[j] * sigm(gg[j]);
      d_store<VEC>(dst + c, b);
    }
  }
}

// ---- decode ---------------------------------------------------------------------------------------------------------
constexpr int DCT = 256;

// One token per sequence; VEC columns per thread. KEEP: rows of the state a thread holds between its two uses (0: read twice).
template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(DCT) gdelta_decode_kernel(const DeltaParams p) {
  extern __shared__ __align__(16) float dsm[];   // w | u | a u | r [D each] | x [rank] | seen [V] | sums [groups][V]
  __shared__ float red[32];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const long long t = p.cu[b];
  if (p.cu[b + 1] <= t) return;
  const int D = p.D, V = p.V, HD = h * D, rank = p.rank;
  float *sw = dsm, *su = dsm + D, *sb = dsm + 2 * D, *sr = dsm + 3 * D, *sx = dsm + 4 * D, *seen = sx + rank, *sums = seen + V;
  const int vcols = V / VEC, groups = max(1, DCT / vcols);
  float* st = p.state + ((long long)(p.slots ? p.slots[b] : b) * p.H + h) * (long long)D * V;

  // the state is on its way while the gates are formed
  const int cg = tid % vcols, rg = tid / vcols;
  const bool on = KEEP && rg < groups;
  float s[KEEP ? KEEP : 1][VEC];
  if constexpr (KEEP > 0) {
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      const int d = rg + i * groups;
      if (on && d < D) d_load<VEC>(st + (long long)d * V + cg * VEC, s[i]);
    }
  }
  const T* x = reinterpret_cast<const T*>(p.x) + t * p.ld;
  for (int i = tid; i < rank; i += DCT) sx[i] = tanhf(d_of(x[i]));
  const T* k = reinterpret_cast<const T*>(p.k) + t * p.ld + HD;
  float ss = 0.f;
  for (int d = tid; d < D; d += DCT) {
    const float kv = d_of(k[d]);
    su[d] = kv;
    ss += kv * kv;
  }
  const float len = sqrtf(block_sum(ss, red) + p.unit_eps), inv = 1.f / len;      // its barriers also publish sx and su
  // low-rank products: a few adjacent lanes share a channel
  const T* w2 = reinterpret_cast<const T*>(p.w2) + (long long)HD * rank;
  const bool vec2 = rank % 4 == 0 && (reinterpret_cast<uintptr_t>(p.w2) & 15) == 0;
  int share = 1;
  while (share < 32 && 2 * share * D <= DCT) share <<= 1;
  for (int d0 = 0; d0 < D; d0 += DCT / share) {      // the same rounds for every lane
    const int d = d0 + tid / share, sub = tid % share;
    float z = 0.f;
    if (d < D) {
      const T* m = w2 + (long long)d * rank;
      if (vec2) {
#pragma unroll 4
        for (int i = sub * 4; i < rank; i += share * 4) {
          float c[4];
          d_load<4>(m + i, c);
          z += (c[0] * sx[i] + c[1] * sx[i + 1]) + (c[2] * sx[i + 2] + c[3] * sx[i + 3]);
        }
      } else {
        for (int i = sub; i < rank; i += share) z += d_of(m[i]) * sx[i];
      }
    }
    for (int o = share >> 1; o > 0; o >>= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
    if (d < D && sub == 0) {
      const float u = su[d] * inv;
      sw[d] = expf(-p.rate * sigm(z + p.w0[HD + d]));
      su[d] = u;
      sb[d] = sigm(d_of(reinterpret_cast<const T*>(p.a)[t * p.ld + HD + d]) + p.a0[HD + d]) * u;
      sr[d] = d_of(reinterpret_cast<const T*>(p.r)[t * p.ld + HD + d]);
    }
  }
  __syncthreads();
  const T* vrow = reinterpret_cast<const T*>(p.v) + t * p.ld + (long long)h * V;
  // u^T S: partial sums of the row groups, then of the columns
  for (int q = tid; q < vcols * groups; q += DCT) {      // one round unless V / VEC > DCT
    const int c = q % vcols, g = q / vcols;
    float acc[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) acc[j] = 0.f;
    if constexpr (KEEP > 0) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i) {
        const int d = g + i * groups;
        if (d < D)
#pragma unroll
          for (int j = 0; j < VEC; ++j) acc[j] = fmaf(su[d], s[i][j], acc[j]);
      }
    } else {
      for (int d = g; d < D; d += groups) {
        float a[VEC];
        d_load<VEC>(st + (long long)d * V + c * VEC, a);
#pragma unroll
        for (int j = 0; j < VEC; ++j) acc[j] = fmaf(su[d], a[j], acc[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) sums[g * V + c * VEC + j] = acc[j];
  }
  __syncthreads();
  for (int c = tid; c < V; c += DCT) {
    float y = 0.f;
    for (int g = 0; g < groups; ++g) y += sums[g * V + c];
    seen[c] = y;
  }
  __syncthreads();
  for (int q = tid; q < vcols * groups; q += DCT) {
    const int c = q % vcols, g = q / vcols;
    float acc[VEC], v[VEC], y[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      acc[j] = 0.f;
      v[j] = d_of(vrow[c * VEC + j]) * len;
      y[j] = seen[c * VEC + j];
    }
    auto update = [&](int d, float (&a)[VEC]) {
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        a[j] = fmaf(sb[d], -y[j], fmaf(sw[d], a[j], su[d] * v[j]));
        acc[j] = fmaf(sr[d], a[j], acc[j]);
      }
      d_store<VEC>(st + (long long)d * V + c * VEC, a);
    };
    if constexpr (KEEP > 0) {
#pragma unroll
      for (int i = 0; i < KEEP; ++i)
        if (g + i * groups < D) update(g + i * groups, s[i]);
    } else {
      for (int d = g; d < D; d += groups) {
        float a[VEC];
        d_load<VEC>(st + (long long)d * V + c * VEC, a);
        update(d, a);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) sums[g * V + c * VEC + j] = acc[j];
  }
  __syncthreads();
  ss = 0.f;
  for (int c = tid; c < V; c += DCT) {
    float y = 0.f;
    for (int g = 0; g < groups; ++g) y += sums[g * V + c];
    seen[c] = y;                                  // this thread's own columns
    ss += y * y;
  }
  const float f = p.scale / sqrtf(block_sum(ss, red) / (float)V + p.eps);
  const T* g = reinterpret_cast<const T*>(p.g) + t * p.ld + (long long)h * V;
  T* out = reinterpret_cast<T*>(p.out) + t * p.ld_out + (long long)h * V;
  for (int c = tid; c < V; c += DCT) d_put(out + c, seen[c] * f * p.norm[h * V + c] * sigm(d_of(g[c])));
}

// out [rows, n] = tanh(x) of columns at pitch ld
template <typename T>
__global__ void tanh_rows_kernel(const T* __restrict__ x, long long ld, T* __restrict__ out, int rows, int n) {
  const long long total = (long long)rows * n;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / n;
    d_put(out + i, tanhf(d_of(x[r * ld + (i - r * n)])));
  }
}

bool al(const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

int lanes_for(int n, int vec) {
  int l = 1;
  while (l < 32 && l * vec < n) l <<= 1;
  return l;
}

int row_blocks(long long items, int lanes) {
  const long long b = (items + RT / lanes - 1) / (RT / lanes), cap = (long long)sm_count() * 16;
  return (int)(b < cap ? b : cap);
}

template <int DP, int RPT, int CPT, int NT>
int launch_scan(const DeltaParams& p, cudaStream_t s) {
  using C = ScanCfg<DP, RPT, CPT, NT>;
  constexpr int SMEM = 2 * C::STAGE * 4;
  auto kern = gdelta_scan_kernel<DP, RPT, CPT, NT>;
  if constexpr (SMEM > 48 * 1024) {
    static bool attr_set[64] = {false};
    int dev = 0;
    cudaGetDevice(&dev);
    if (dev < 0 || dev >= 64) dev = 0;
    if (!attr_set[dev]) {
      if (check_cuda(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM),
                     "cudaFuncSetAttribute(gdelta_scan)"))
        return -1;
      attr_set[dev] = true;
    }
  }
  kern<<<dim3((p.V + C::CT - 1) / C::CT, p.H, p.B), NT, SMEM, s>>>(p);
  return check_cuda(cudaGetLastError(), "gdelta_scan launch");
}

template <typename T>
int run_scan(DeltaParams& p, cudaStream_t s) {
  const int vec = p.vec ? 4 : 1, lanes = lanes_for(p.D, vec);
  const int blocks = row_blocks((long long)p.T * p.H, lanes);
  if (p.vec) gdelta_rows_kernel<T, 4><<<blocks, RT, 0, s>>>(p, lanes);
  else gdelta_rows_kernel<T, 1><<<blocks, RT, 0, s>>>(p, lanes);
  if (check_cuda(cudaGetLastError(), "gdelta_rows launch")) return -1;
  // one column per thread while the GPU is not full of warps (the shortest wait per token), else more
  const long long warps = (long long)p.B * p.H * p.V * (p.D <= 64 ? 4 : p.D <= 128 ? 8 : 16) / 32;
  const int cols = warps <= 4LL * sm_count() ? 1 : warps <= 8LL * sm_count() ? 2 : 4;
#define EDL_GS(DP, RPT, NT_)                                        \
  return cols == 1 ? launch_scan<DP, RPT, 1, NT_>(p, s) : cols == 2 \
             ? launch_scan<DP, RPT, 2, NT_>(p, s) : launch_scan<DP, RPT, 4, NT_>(p, s)
  if (p.D <= 32) EDL_GS(32, 8, 64);
  if (p.D <= 64) EDL_GS(64, 16, 64);
  if (p.D <= 128) EDL_GS(128, 16, 64);
  if (p.D <= 256) return launch_scan<256, 16, 2, 128>(p, s);
  return launch_scan<512, 16, 2, 128>(p, s);
#undef EDL_GS
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

// o [T, H * V] fp32 (no output norm); r, k, a [T, H * D], v [T, H * V]: columns of a projection at pitch ld; z [T, H * D] fp32;
// rows: workspace [T, H, 4 D + V] fp32.
EDL_HOST_API int edl_gdelta_scan(const void* r, const void* k, const void* v, const void* a, int f32, long long ld,
                                 const float* z, const float* w0, const float* a0, float rate, float unit_eps,
                                 const int* cu, const int* slots, float* state, float* o, float* rows, int T, int B, int H,
                                 int D, int V, void* stream) {
  if (B <= 0 || T <= 0) return 0;
  if (bad_sizes("edl_gdelta_scan", B, H, D, V)) return -1;
  DeltaParams p{};
  p.r = r; p.k = k; p.v = v; p.a = a; p.ld = ld; p.z = z; p.w0 = w0; p.a0 = a0; p.rate = rate; p.unit_eps = unit_eps;
  p.cu = cu; p.slots = slots; p.state = state; p.o = o; p.rows = rows; p.T = T; p.B = B; p.H = H; p.D = D; p.V = V;
  const size_t n = f32 ? 16 : 8;
  p.vec = D % 4 == 0 && V % 4 == 0 && ld % 4 == 0 && al(r, n) && al(k, n) && al(v, n) && al(a, n) && al(z, 16) &&
          al(w0, 16) && al(a0, 16) && al(rows, 16);
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? run_scan<float>(p, s) : run_scan<__nv_bfloat16>(p, s);
}

// out [T, H * V] (operand type, pitch ld_out) = rms_norm of each head of o * norm * sigmoid(g) * scale.
EDL_HOST_API int edl_gdelta_finish(const float* o, const void* g, int f32, long long ld, const float* norm, float eps,
                                   float scale, void* out, long long ld_out, int T, int H, int V, void* stream) {
  if (T <= 0) return 0;
  DeltaParams p{};
  p.o = const_cast<float*>(o); p.g = g; p.ld = ld; p.norm = norm; p.eps = eps; p.scale = scale; p.out = out;
  p.ld_out = ld_out; p.T = T; p.H = H; p.V = V;
  const size_t n = f32 ? 16 : 8;
  const bool vec = V % 4 == 0 && ld % 4 == 0 && ld_out % 4 == 0 && al(o, 16) && al(g, n) && al(norm, 16) && al(out, n);
  const int lanes = lanes_for(V, vec ? 4 : 1), blocks = row_blocks((long long)T * H, lanes);
  cudaStream_t s = (cudaStream_t)stream;
  if (f32) {
    if (vec) gdelta_finish_kernel<float, 4><<<blocks, RT, 0, s>>>(p, lanes);
    else gdelta_finish_kernel<float, 1><<<blocks, RT, 0, s>>>(p, lanes);
  } else {
    if (vec) gdelta_finish_kernel<__nv_bfloat16, 4><<<blocks, RT, 0, s>>>(p, lanes);
    else gdelta_finish_kernel<__nv_bfloat16, 1><<<blocks, RT, 0, s>>>(p, lanes);
  }
  return check_cuda(cudaGetLastError(), "gdelta_finish launch");
}

// One token per sequence (row cu[b] of the projection), low-rank product w2 [H * D, rank] tanh(x [rank]), output norm and gate
// included; out in the projection's type at pitch ld_out.
EDL_HOST_API int edl_gdelta_decode(const void* r, const void* k, const void* v, const void* a, const void* g, const void* x,
                                   int f32, long long ld, const void* w2, int rank, const float* w0, const float* a0,
                                   float rate, float unit_eps, const int* cu, const int* slots, float* state,
                                   const float* norm, float eps, float scale, void* out, long long ld_out, int B, int H,
                                   int D, int V, void* stream) {
  if (B <= 0) return 0;
  if (bad_sizes("edl_gdelta_decode", B, H, D, V)) return -1;
  if (!state || rank < 0 || rank > 4096) {
    set_last_error("edl_gdelta_decode: needs a state pool and a rank up to 4096 (rank=%d)", rank);
    return -1;
  }
  DeltaParams p{};
  p.r = r; p.k = k; p.v = v; p.a = a; p.g = g; p.x = x; p.ld = ld; p.w2 = w2; p.rank = rank; p.w0 = w0; p.a0 = a0;
  p.rate = rate; p.unit_eps = unit_eps; p.cu = cu; p.slots = slots; p.state = state; p.norm = norm; p.eps = eps;
  p.scale = scale; p.out = out; p.ld_out = ld_out; p.B = B; p.H = H; p.D = D; p.V = V;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = V % 4 == 0 && al(state, 16);
  const int vcols = v4 ? V / 4 : V;
  const int groups = vcols >= DCT ? 1 : DCT / vcols;
  const int rows = vcols <= DCT ? (D + groups - 1) / groups : 17;
  const size_t smem = (size_t)(4 * D + rank + V + groups * V) * sizeof(float);     // <= 2048 + 4096 + 1024 + 1024 floats
  const dim3 grid(H, B);
#define EDL_GD(TT, V_, K_) gdelta_decode_kernel<TT, V_, K_><<<grid, DCT, smem, s>>>(p)
#define EDL_GDH(TT, V_)                \
  if (rows <= 4) EDL_GD(TT, V_, 4);    \
  else if (rows <= 8) EDL_GD(TT, V_, 8);  \
  else if (rows <= 16) EDL_GD(TT, V_, 16); \
  else EDL_GD(TT, V_, 0)
  if (f32) {
    if (v4) { EDL_GDH(float, 4); } else { EDL_GDH(float, 1); }
  } else {
    if (v4) { EDL_GDH(__nv_bfloat16, 4); } else { EDL_GDH(__nv_bfloat16, 1); }
  }
#undef EDL_GDH
#undef EDL_GD
  return check_cuda(cudaGetLastError(), "gdelta_decode launch");
}

// out [rows, n] = tanh(x), x at pitch ld, in the operand type.
EDL_HOST_API int edl_tanh_rows(const void* x, int f32, long long ld, void* out, int rows, int n, void* stream) {
  if (rows <= 0 || n <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const long long want = ((long long)rows * n + 255) / 256, cap = (long long)sm_count() * 8;
  const int blocks = (int)(want < cap ? want : cap);
  if (f32) tanh_rows_kernel<float><<<blocks, 256, 0, s>>>((const float*)x, ld, (float*)out, rows, n);
  else tanh_rows_kernel<__nv_bfloat16><<<blocks, 256, 0, s>>>((const __nv_bfloat16*)x, ld, (__nv_bfloat16*)out, rows, n);
  return check_cuda(cudaGetLastError(), "tanh_rows launch");
}
