// Element-wise and row kernels around an fp32 residual stream.
//
// Models that keep the sum of their branches in 32 bits hold x [T, W] as fp32; every branch reads it through a norm
// that writes the operand of the next product (bf16, or fp32 for an all-fp32 model) and its output projection
// accumulates straight into x. The kernels here are what sits between those products:
//
//   * embedding rows into the stream (and, for models whose passes read [x ; x0], into the right half of that operand);
//   * RMS norm, optionally followed by a token shift (each row is blended with the normalised row before it; the row
//     before a step's first row lives in a per-slot state that the same launch brings up to date);
//   * the left half of a pass's [x ; x0] operand;
//   * xIELU, a two-branch activation with two learned numbers;
//   * the attention prologue: per-head RMS norm of q and k, position-dependent query temperature and the page append,
//     in one pass over the packed projection;
//   * the same with biases, optional norms over all query heads (all key heads) at once, rotated halves or neighbours, and values that
//     blend with another layer's;
//   * a branch that is normed (and scaled per channel) before it joins the stream, with the norm that reads the sum;
//   * gated units in 32 bits or at odd sizes, and scaled and soft-capped logits.
//
// Compiled without fast-math: these are the parts of such a model that are computed in 32 bits.
#include "common.cuh"

#include <type_traits>

namespace edl {
namespace {

template <typename T>
__device__ __forceinline__ float ld1(const T* p);
template <>
__device__ __forceinline__ float ld1<float>(const float* p) { return *p; }
template <>
__device__ __forceinline__ float ld1<__nv_bfloat16>(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <int VEC, typename T>
__device__ __forceinline__ void ldv(const T* p, float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
  } else if constexpr (VEC == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = unpack_bf16x2(a.x), hi = unpack_bf16x2(a.y);
    v[0] = lo.x; v[1] = lo.y; v[2] = hi.x; v[3] = hi.y;
  } else if constexpr (VEC == 8 && sizeof(T) == 2) {
    const uint4 a = *reinterpret_cast<const uint4*>(p);
    const uint32_t w[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 f = unpack_bf16x2(w[i]);
      v[2 * i] = f.x;
      v[2 * i + 1] = f.y;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = ld1<T>(p + i);
  }
}
template <int VEC, typename T>
__device__ __forceinline__ void stv(T* p, const float (&v)[VEC]) {
  if constexpr (VEC == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (VEC == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
  } else if constexpr (VEC == 8 && sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]),
                                              pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) st1(p + i, v[i]);
  }
}

// Largest b with cu[b] <= r (cu is a non-decreasing prefix sum).
__device__ __forceinline__ int seq_of_row(const int* cu, int nseq, int r) {
  int lo = 0, hi = nseq;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= r) lo = mid; else hi = mid;
  }
  return lo;
}

// ---- embedding -------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void embed_stream_kernel(const T* __restrict__ table, const long long* __restrict__ ids, float scale,
                                    float* __restrict__ x, T* __restrict__ right, long long ld_right, int rows, int W,
                                    int V, int* status) {
  const int per = W / VEC;
  const long long total = (long long)rows * per;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total;
       i += (long long)gridDim.x * blockDim.x) {
    const int r = (int)(i / per), c = (int)(i - (long long)r * per) * VEC;
    const long long id = ids[r];
    float v[VEC];
    if (id < 0 || id >= V) {
      if (status) atomicCAS(status, 0, EDL_BAD_INDEX);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    } else {
      ldv<VEC>(table + id * W + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= scale;
    }
    stv<VEC>(x + (long long)r * W + c, v);
    if (right) stv<VEC>(right + r * ld_right + c, v);
  }
}

// ---- left half of [x ; x0] -------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void cast_rows_kernel(const float* __restrict__ x, T* __restrict__ out, long long ld_out, int rows, int W) {
  const int per = W / VEC;
  const long long total = (long long)rows * per;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total;
       i += (long long)gridDim.x * blockDim.x) {
    const int r = (int)(i / per), c = (int)(i - (long long)r * per) * VEC;
    float v[VEC];
    ldv<VEC>(x + (long long)r * W + c, v);
    stv<VEC>(out + r * ld_out + c, v);
  }
}

// ---- RMS norm (+ token shift) -----------------------------------------------------------------------------------
constexpr int NT = 256;

// Two block-wide sums at once.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
  const int lane = threadIdx.x & 31, w = threadIdx.x >> 5;
  a = warp_sum(a);
  b = warp_sum(b);
  __syncthreads();
  if (lane == 0) red[w] = make_float2(a, b);
  __syncthreads();
  float2 t = red[0];
#pragma unroll
  for (int i = 1; i < NT / 32; ++i) {
    t.x += red[i].x;
    t.y += red[i].y;
  }
  return t;
}

// Many rows, a whole row in registers: a CTA walks `per` consecutive rows and keeps the normalised row before the
// current one, so each row is read once (plus the one in front of the CTA's first).
template <typename TO, int NV>
__global__ void __launch_bounds__(NT)
norm_shift_rows_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ mu, float eps,
                       int rows, int W, const int* __restrict__ cu, int nseq, const int* __restrict__ slots,
                       float* __restrict__ state, long long ld_state, float offset, TO* __restrict__ out, int per) {
  __shared__ float2 red[NT / 32];
  constexpr int STEP = NT * 4;
  const int r0 = blockIdx.x * per, r1 = min(rows, r0 + per);
  const float inv_w = 1.f / (float)W;
  int b = mu ? seq_of_row(cu, nseq, r0) : 0;
  float wv[NV][4], mv[NV][4], h[NV][4], before[NV][4], next[NV][4];
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int c = threadIdx.x * 4 + k * STEP;
    if (c < W) {
      ldv<4>(w + c, wv[k]);
#pragma unroll
      for (int j = 0; j < 4; ++j) wv[k][j] += offset;
      if (mu) ldv<4>(mu + c, mv[k]);
    }
  }
  auto load = [&](int r, float (&d)[NV][4]) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * 4 + k * STEP;
      if (c < W) ldv<4>(x + (long long)r * W + c, d[k]);
    }
  };
  // h = rms_norm of the row in d
  auto norm = [&](const float (&d)[NV][4]) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k)
      if (threadIdx.x * 4 + k * STEP < W)
#pragma unroll
        for (int j = 0; j < 4; ++j) s += d[k][j] * d[k][j];
    const float rs = 1.f / sqrtf(block_sum2(s, 0.f, red).x * inv_w + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) h[k][j] = d[k][j] * rs * wv[k][j];
  };
  if (mu && r0 > cu[b]) {
    load(r0 - 1, next);
    norm(next);
#pragma unroll
    for (int k = 0; k < NV; ++k)
#pragma unroll
      for (int j = 0; j < 4; ++j) before[k][j] = h[k][j];
  }
  load(r0, next);
  for (int r = r0; r < r1; ++r) {
    norm(next);
    if (r + 1 < r1) load(r + 1, next);
    float* st = nullptr;
    int last = -1;
    if (mu) {
      while (b + 1 < nseq && r >= cu[b + 1]) ++b;
      if (r == cu[b]) {                 // first row of a sequence: the row before it is the slot's state, or zeros
        st = state ? state + (long long)slots[b] * ld_state : nullptr;
        last = cu[b + 1] - 1;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
          const int c = threadIdx.x * 4 + k * STEP;
#pragma unroll
          for (int j = 0; j < 4; ++j) before[k][j] = 0.f;
          if (st && c < W) ldv<4>(st + c, before[k]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * 4 + k * STEP;
      if (c < W) {
        float o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j] = mu ? h[k][j] + (before[k][j] - h[k][j]) * mv[k][j] : h[k][j];
        stv<4>(out + (long long)r * W + c, o);
        if (st && last == r) stv<4>(st + c, h[k]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) before[k][j] = h[k][j];
    }
    if (st && last != r) {              // the state's only reader also leaves the step's last row in it
      float s = 0.f, v[4];
      const float* xl = x + (long long)last * W;
      for (int c = threadIdx.x * 4; c < W; c += STEP) {
        ldv<4>(xl + c, v);
#pragma unroll
        for (int j = 0; j < 4; ++j) s += v[j] * v[j];
      }
      const float rl = 1.f / sqrtf(block_sum2(s, 0.f, red).x * inv_w + eps);
#pragma unroll
      for (int k = 0; k < NV; ++k) {
        const int c = threadIdx.x * 4 + k * STEP;
        if (c < W) {
          ldv<4>(xl + c, v);
#pragma unroll
          for (int j = 0; j < 4; ++j) v[j] = v[j] * rl * wv[k][j];
          stv<4>(st + c, v);
        }
      }
    }
  }
}

// One CTA per row. NV: vectors of VEC elements each thread keeps of a row (0: rows too wide for registers are read
// twice). Without `mu` this is a plain norm.
template <typename TO, int VEC, int NV>
__global__ void __launch_bounds__(NT)
norm_shift_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ mu, float eps,
                  int rows, int W, const int* __restrict__ cu, int nseq, const int* __restrict__ slots,
                  float* __restrict__ state, long long ld_state, float offset, TO* __restrict__ out) {
  __shared__ float2 red[NT / 32];
  const int r = blockIdx.x;
  const float inv_w = 1.f / (float)W;
  const float* xr = x + (long long)r * W;
  const float* xp = nullptr;   // the row before, when this step brought it
  float* st = nullptr;
  int last = -1;
  if (mu) {
    const int b = seq_of_row(cu, nseq, r);
    if (r > cu[b]) {
      xp = xr - W;
    } else if (state) {
      st = state + (long long)slots[b] * ld_state;
      last = cu[b + 1] - 1;
    }
  }
  constexpr int STEP = NT * VEC;
  constexpr int KEEP = NV > 0 ? NV : 1;
  float a[KEEP][VEC], p[KEEP][VEC];
  float sa = 0.f, sp = 0.f;
  if constexpr (NV > 0) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * VEC + k * STEP;
      if (c < W) {
        ldv<VEC>(xr + c, a[k]);
        if (xp) ldv<VEC>(xp + c, p[k]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          sa += a[k][j] * a[k][j];
          if (xp) sp += p[k][j] * p[k][j];
        }
      }
    }
  } else {
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(xr + c, a[0]);
      if (xp) ldv<VEC>(xp + c, p[0]);
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        sa += a[0][j] * a[0][j];
        if (xp) sp += p[0][j] * p[0][j];
      }
    }
  }
  const float2 s = block_sum2(sa, sp, red);
  const float ra = 1.f / sqrtf(s.x * inv_w + eps), rp = 1.f / sqrtf(s.y * inv_w + eps);
  auto emit = [&](int c, const float (&av)[VEC], const float (&pv)[VEC]) {
    float wv[VEC], h[VEC];
    ldv<VEC>(w + c, wv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      wv[j] += offset;
      h[j] = av[j] * ra * wv[j];
    }
    if (mu) {
      float m[VEC], before[VEC], o[VEC];
      ldv<VEC>(mu + c, m);
      if (st) {
        ldv<VEC>(st + c, before);
      } else {
#pragma unroll
        for (int j = 0; j < VEC; ++j) before[j] = xp ? pv[j] * rp * wv[j] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = h[j] + (before[j] - h[j]) * m[j];
      stv<VEC>(out + (long long)r * W + c, o);
      if (st && last == r) stv<VEC>(st + c, h);
    } else {
      stv<VEC>(out + (long long)r * W + c, h);
    }
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * VEC + k * STEP;
      if (c < W) emit(c, a[k], p[k]);
    }
  } else {
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(xr + c, a[0]);
      if (xp) ldv<VEC>(xp + c, p[0]);
      emit(c, a[0], p[0]);
    }
  }
  if (st && last != r) {
    // The CTA of a sequence's first row is the only reader of its state; having read it, it also normalises the last
    // row and leaves that one for the next step. Nobody else touches the state, so no launch has to follow.
    const float* xl = x + (long long)last * W;
    float sl = 0.f, v[VEC], wv[VEC];
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(xl + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sl += v[j] * v[j];
    }
    const float rl = 1.f / sqrtf(block_sum2(sl, 0.f, red).x * inv_w + eps);
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(xl + c, v);
      ldv<VEC>(w + c, wv);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = v[j] * rl * (wv[j] + offset);
      stv<VEC>(st + c, v);
    }
  }
}

// ---- RMS norm over the heads of a [T, H * V] matrix with one weight vector for all heads ------------------------------
template <typename TO>
__global__ void __launch_bounds__(NT)
head_norm_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps, long long items, int V,
                 TO* __restrict__ out) {
  const int lane = threadIdx.x & 31;
  const long long stride = (long long)gridDim.x * (NT / 32);
  for (long long it = blockIdx.x * (long long)(NT / 32) + (threadIdx.x >> 5); it < items; it += stride) {
    const float* src = o + it * V;
    float s = 0.f;
    for (int c = lane; c < V; c += 32) s += src[c] * src[c];
    s = warp_sum(s);
    const float rs = 1.f / sqrtf(s / (float)V + eps);
    for (int c = lane; c < V; c += 32) st1(out + it * V + c, src[c] * rs * w[c]);
  }
}

// ---- xIELU ------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float softplus1(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <typename T, int VEC>
__global__ void xielu_kernel(const T* __restrict__ z, const float* __restrict__ act, T* __restrict__ y,
                             long long n_vec) {
  const float ap = softplus1(act[0]), an = 0.5f + softplus1(act[1]);
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < n_vec;
       i += (long long)gridDim.x * blockDim.x) {
    float v[VEC];
    ldv<VEC>(z + i * VEC, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float t = v[j];
      float e;   // e^t - 1 - t for t <= 0
      if constexpr (sizeof(T) == 4) {
        e = expm1f(t) - t;
      } else {   // the operand has 8 bits: a short Taylor sum near zero, the hardware exponential elsewhere
        const float near = 0.5f * t * t * fmaf(t * (1.f / 3.f), fmaf(t, 0.25f, 1.f), 1.f);
        e = t > -0.06f ? near : __expf(t) - 1.f - t;
      }
      v[j] = t > 0.f ? ap * t * t + 0.5f * t : an * e + 0.5f * t;
    }
    stv<VEC>(y + i * VEC, v);
  }
}

// ---- attention prologue -------------------------------------------------------------------------------------------------
// qkv [T, ld]: Hq query heads of D, Hkv key heads of D, Hkv value heads of Dv. One warp per (token, head): q and k are
// RMS-normed over D (weights may be null: no norm), q is multiplied by its position's temperature
// 1 + coef * ln(floor((p + 1) / every) + 1) (every <= 0: none) and written to q_out; k and v go to their page slot.
template <typename T, int VEC>
__global__ void __launch_bounds__(NT)
qkv_prologue_kernel(const T* __restrict__ qkv, long long ld, const int* __restrict__ pos,
                    const int* __restrict__ slots, const float* __restrict__ qw, const float* __restrict__ kw,
                    float eps, float coef, float every, int T_rows, int Hq, int Hkv, int D, int Dv,
                    T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages, long long ld_kpage,
                    long long ld_vpage, long long num_slots, int* status) {
  const int lane = threadIdx.x & 31;
  const int heads = Hq + 2 * Hkv;
  const long long items = (long long)T_rows * heads;
  const long long stride = (long long)gridDim.x * (NT / 32);
  for (long long it = blockIdx.x * (long long)(NT / 32) + (threadIdx.x >> 5); it < items; it += stride) {
    const int t = (int)(it / heads), h = (int)(it - (long long)t * heads);
    const T* row = qkv + t * ld;
    const int hk = h < Hq ? -1 : (h < Hq + Hkv ? h - Hq : h - Hq - Hkv);
    long long slot = 0;
    if (h >= Hq) {
      slot = slots[t];
      if (slot < 0) continue;
      if (slot >= num_slots) {
        if (status) atomicCAS(status, 0, EDL_BAD_INDEX);
        continue;
      }
    }
    if (h >= Hq + Hkv) {   // value head: copied
      const T* src = row + (long long)(Hq + Hkv) * D + (long long)hk * Dv;
      T* dst = v_pages + slot * ld_vpage + (long long)hk * Dv;
      for (int c = lane * VEC; c < Dv; c += 32 * VEC) {
        float v[VEC];
        ldv<VEC>(src + c, v);
        stv<VEC>(dst + c, v);
      }
      continue;
    }
    const bool is_q = h < Hq;
    const T* src = row + (long long)h * D;          // key heads follow the query heads
    const float* w = is_q ? qw : kw;
    float scale = 1.f;
    if (w) {
      float s = 0.f;
      for (int c = lane * VEC; c < D; c += 32 * VEC) {
        float v[VEC];
        ldv<VEC>(src + c, v);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s += v[j] * v[j];
      }
      s = warp_sum(s);
      scale = 1.f / sqrtf(s / (float)D + eps);
    }
    float temp = 1.f;
    if (is_q && every > 0.f) temp = 1.f + coef * logf(floorf(((float)pos[t] + 1.f) / every) + 1.f);
    T* dst = is_q ? q_out + ((long long)t * Hq + h) * D : k_pages + slot * ld_kpage + (long long)hk * D;
    for (int c = lane * VEC; c < D; c += 32 * VEC) {
      float v[VEC], wv[VEC];
      ldv<VEC>(src + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) wv[j] = w ? w[c + j] : 1.f;
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] = v[j] * scale * wv[j] * temp;
      stv<VEC>(dst + c, v);
    }
  }
}

// The same for heads of up to 128 elements in 4-element pieces: a lane holds its piece of four heads at a time in
// registers, so that four rows are in flight per warp and nothing is read twice.
template <typename T>
__global__ void __launch_bounds__(NT)
qkv_prologue_small_kernel(const T* __restrict__ qkv, long long ld, const int* __restrict__ pos,
                          const int* __restrict__ slots, const float* __restrict__ qw, const float* __restrict__ kw,
                          float eps, float coef, float every, int T_rows, int Hq, int Hkv, int D, int Dv,
                          T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages, long long ld_kpage,
                          long long ld_vpage, long long num_slots, int* status) {
  constexpr int U = 4;
  const int lane = threadIdx.x & 31, c = lane * 4;
  const int heads = Hq + 2 * Hkv, per_token = (heads + U - 1) / U;
  const bool in_d = c < D, in_v = c < Dv;
  float wq[4] = {1.f, 1.f, 1.f, 1.f}, wk[4] = {1.f, 1.f, 1.f, 1.f};
  if (in_d) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (qw) wq[j] = qw[c + j];
      if (kw) wk[j] = kw[c + j];
    }
  }
  const float inv_d = 1.f / (float)D;
  const unsigned groups = (unsigned)T_rows * per_token, stride = gridDim.x * (NT / 32);
  for (unsigned it = blockIdx.x * (NT / 32) + (threadIdx.x >> 5); it < groups; it += stride) {
    const int t = it / per_token, h0 = (it - t * per_token) * U;
    const T* row = qkv + t * ld;
    float v[U][4], s[U];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int h = h0 + u;
      const bool val = h >= Hq + Hkv;
      s[u] = 0.f;
      if (h < heads && (val ? in_v : in_d)) {
        ldv<4>(row + (val ? (Hq + Hkv) * D + (h - Hq - Hkv) * Dv : h * D) + c, v[u]);
        s[u] = v[u][0] * v[u][0] + v[u][1] * v[u][1] + v[u][2] * v[u][2] + v[u][3] * v[u][3];
      }
    }
    long long slot = 0;
    float temp = 1.f;
    if (h0 + U > Hq) {
      slot = slots[t];
      if (slot >= num_slots) {
        if (status) atomicCAS(status, 0, EDL_BAD_INDEX);
        slot = -1;
      }
    }
    if (h0 < Hq && every > 0.f) temp = 1.f + coef * logf(floorf(((float)pos[t] + 1.f) / every) + 1.f);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int u = 0; u < U; ++u) s[u] += __shfl_xor_sync(0xffffffffu, s[u], o);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int h = h0 + u;
      if (h >= heads) break;
      if (h < Hq) {
        const float r = (qw ? 1.f / sqrtf(s[u] * inv_d + eps) : 1.f) * temp;
#pragma unroll
        for (int j = 0; j < 4; ++j) v[u][j] *= r * wq[j];
        if (in_d) stv<4>(q_out + ((long long)t * Hq + h) * D + c, v[u]);
      } else if (slot >= 0 && h < Hq + Hkv) {
        const float r = kw ? 1.f / sqrtf(s[u] * inv_d + eps) : 1.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) v[u][j] *= r * wk[j];
        if (in_d) stv<4>(k_pages + slot * ld_kpage + (h - Hq) * D + c, v[u]);
      } else if (slot >= 0) {
        if (in_v) stv<4>(v_pages + slot * ld_vpage + (h - Hq - Hkv) * Dv + c, v[u]);
      }
    }
  }
}

// ---- attention prologue with full-width norms and rotation -----------------------------------------------------------------
constexpr int RP_MAX_PAIRS = 512;     // rotated pairs of a head

struct RotaryPrologueParams {
  long long ld;
  const int* pos;
  const int* slots;
  const float *qw, *kw;      // [Hq * D], [Hkv * D], or null: no norm
  float eps;
  const float* freq;         // [pairs] leading parts of the frequencies, then [pairs] the parts below their last bit
  int pairs, Hq, Hkv, D, Dv;
  long long ld_kpage, ld_vpage, num_slots;
  int* status;
  int neighbours;            // elements 2j and 2j + 1 form a pair (else j and j + pairs)
  float mag;                 // factor of cosines and sines
  const float* bias;         // [Hq * D + Hkv * (D + Dv)] added to the row first, or null
  const void* v_first;       // values [T, Hkv * Dv] at pitch ld_first to blend in by *lam, or null
  long long ld_first;
  const float* lam;
};

// cos and sin of position * frequency i, times mag. Angles are as exact as in the latent prologue: the product's rounding
// error and the frequency's own are a small second rotation.
__device__ __forceinline__ float2 turn_of(const RotaryPrologueParams& p, float fp, int i) {
  const float f = p.freq[i], a = fp * f;
  const float e = fmaf(fp, f, -a) + fp * p.freq[p.pairs + i];
  float s, c;
  sincosf(a, &s, &c);
  const float ce = 1.f - 0.5f * e * e, se = e - e * e * e * (1.f / 6.f);
  return make_float2((c * ce - s * se) * p.mag, (s * ce + c * se) * p.mag);
}

template <int VEC>
__device__ __forceinline__ void ldw(const float* w, float (&v)[VEC]) {
  if constexpr (VEC % 4 == 0) {
#pragma unroll
    for (int i = 0; i < VEC; i += 4) {
      const float4 a = *reinterpret_cast<const float4*>(w + i);
      v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < VEC; ++i) v[i] = w[i];
  }
}

// v[j] += bias[at + j]
template <int VEC>
__device__ __forceinline__ void add_bias(const float* bias, int at, float (&v)[VEC]) {
  if (!bias) return;
  float b[VEC];
  ldw<VEC>(bias + at, b);
#pragma unroll
  for (int j = 0; j < VEC; ++j) v[j] += b[j];
}

// Values of token t from column c on: bias, blend with the first layer's.
template <typename T, int VEC>
__device__ __forceinline__ void finish_values(const RotaryPrologueParams& p, int t, int c, int at, float (&v)[VEC]) {
  add_bias<VEC>(p.bias, at, v);
  if (p.lam) {
    const float l = *p.lam;
    float f[VEC];
    ldv<VEC>(reinterpret_cast<const T*>(p.v_first) + t * p.ld_first + c, f);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = (1.f - l) * v[j] + l * f[j];
  }
}

// Piece u of a head: VEC elements and their partners (neighbours, unless VEC is 1, are each other's partners within the piece).
// The first `turned` pieces rotate by the cosines cs of their pairs. at: the head's place in the row (for the bias); w, r: norm
// weights of the head and the factor of its norm (w null: no norm).
template <typename T, int VEC>
__device__ __forceinline__ void turn_unit(const RotaryPrologueParams& p, const T* src, T* dst, int at, const float* w, float r,
                                          int u, int turned, const float2* cs) {
  auto load = [&](int c, float (&v)[VEC]) {
    ldv<VEC>(src + c, v);
    add_bias<VEC>(p.bias, at + c, v);
    if (w) {
      float wv[VEC];
      ldw<VEC>(w + c, wv);
#pragma unroll
      for (int j = 0; j < VEC; ++j) v[j] *= r * wv[j];
    }
  };
  float a[VEC];
  if (u >= turned) {
    const int c = 2 * p.pairs + (u - turned) * VEC;
    load(c, a);
    stv<VEC>(dst + c, a);
  } else if (p.neighbours && VEC > 1) {
    const int c = u * VEC;
    load(c, a);
#pragma unroll
    for (int j = 0; j + 1 < VEC; j += 2) {
      const float2 g = cs[(c + j) >> 1];
      const float x = a[j], y = a[j + 1];
      a[j] = x * g.x - y * g.y;
      a[j + 1] = y * g.x + x * g.y;
    }
    stv<VEC>(dst + c, a);
  } else {
    const int c = p.neighbours ? 2 * u : u * VEC, partner = c + (p.neighbours ? 1 : p.pairs);
    float b[VEC];
    load(c, a);
    load(partner, b);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      const float2 g = cs[u * VEC + j];
      const float x = a[j], y = b[j];
      a[j] = x * g.x - y * g.y;
      b[j] = y * g.x + x * g.y;
    }
    stv<VEC>(dst + c, a);
    stv<VEC>(dst + partner, b);
  }
}

// One CTA per token: qkv [T, ld] as above. Queries and keys are RMS-normed over all their heads at once, then the pairs of
// every head turn by position * frequency.
template <typename T, int VEC>
__global__ void __launch_bounds__(NT)
qkv_rotary_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
                  const RotaryPrologueParams p) {
  __shared__ float2 cs[RP_MAX_PAIRS];
  __shared__ float2 red[NT / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  const T* row = qkv + t * p.ld;
  const int nq = p.Hq * p.D, nk = p.Hkv * p.D;
  const float fp = p.pairs ? (float)p.pos[t] : 0.f;
  for (int i = tid; i < p.pairs; i += NT) cs[i] = turn_of(p, fp, i);
  float sq = 0.f, sk = 0.f;
  if (p.qw)
    for (int c = tid * VEC; c < nq; c += NT * VEC) {
      float v[VEC];
      ldv<VEC>(row + c, v);
      add_bias<VEC>(p.bias, c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sq += v[j] * v[j];
    }
  if (p.kw)
    for (int c = tid * VEC; c < nk; c += NT * VEC) {
      float v[VEC];
      ldv<VEC>(row + nq + c, v);
      add_bias<VEC>(p.bias, nq + c, v);
#pragma unroll
      for (int j = 0; j < VEC; ++j) sk += v[j] * v[j];
    }
  const float2 sums = block_sum2(sq, sk, red);       // its barriers also publish cs
  const float rq = p.qw ? 1.f / sqrtf(sums.x / (float)nq + p.eps) : 1.f;
  const float rk = p.kw ? 1.f / sqrtf(sums.y / (float)nk + p.eps) : 1.f;
  long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0, EDL_BAD_INDEX);
    slot = -1;
  }
  const bool inside = p.neighbours && VEC > 1;       // pairs lie within a piece
  const int turned = (inside ? 2 : 1) * p.pairs / VEC;
  const int per = turned + (p.D - 2 * p.pairs) / VEC;   // units of a head: pairs, then the rest
  const int units = (p.Hq + (slot >= 0 ? p.Hkv : 0)) * per;
  for (int i = tid; i < units; i += NT) {
    const int h = i / per, u = i - h * per;
    const bool is_q = h < p.Hq;
    const T* src = row + h * p.D;                    // key heads follow the query heads
    const float* w = is_q ? (p.qw ? p.qw + h * p.D : nullptr) : (p.kw ? p.kw + (h - p.Hq) * p.D : nullptr);
    T* dst = is_q ? q_out + ((long long)t * p.Hq + h) * p.D : k_pages + slot * p.ld_kpage + (h - p.Hq) * p.D;
    turn_unit<T, VEC>(p, src, dst, h * p.D, w, is_q ? rq : rk, u, turned, cs);
  }
  if (slot >= 0)
    for (int c = tid * VEC; c < p.Hkv * p.Dv; c += NT * VEC) {
      float v[VEC];
      ldv<VEC>(row + nq + nk + c, v);
      finish_values<T, VEC>(p, t, c, nq + nk + c, v);
      stv<VEC>(v_pages + slot * p.ld_vpage + c, v);
    }
}

// The same for halves whose units (a piece of VEC elements and its partner) fit KEEP to a thread, without biases and blends: a CTA walks the tokens
// blockIdx.x, blockIdx.x + gridDim.x, ...; norm weights stay in registers, each row is read once, the next one while the
// current one is normed, and cosines and partial sums have two buffers, so that a token costs one barrier.
constexpr int RW_THREADS = 512;

template <typename T, int VEC, int KEEP>
__global__ void __launch_bounds__(RW_THREADS)
qkv_rotary_walk_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
                       const RotaryPrologueParams p, int rows) {
  using Raw = typename std::conditional<sizeof(T) * VEC == 16, uint4, uint2>::type;
  __shared__ float2 cs[2][RP_MAX_PAIRS];
  __shared__ float2 red[2][RW_THREADS / 32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = (blockDim.x + 31) >> 5;
  const int nq = p.Hq * p.D, nk = p.Hkv * p.D, nv = p.Hkv * p.Dv;
  const int turned = p.pairs / VEC, per = turned + (p.D - 2 * p.pairs) / VEC, units = (p.Hq + p.Hkv) * per;
  int col[KEEP];             // first element within the row (< 0: no unit); partner `pairs` further
  bool pair[KEEP];
  float wa[KEEP][VEC], wb[KEEP][VEC];
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int u = tid + i * blockDim.x;
    const int h = u / per, r = u - h * per;
    pair[i] = r < turned;
    col[i] = u < units ? h * p.D + (pair[i] ? r * VEC : 2 * p.pairs + (r - turned) * VEC) : -1;
#pragma unroll
    for (int j = 0; j < VEC; ++j) wa[i][j] = wb[i][j] = 1.f;
    if (col[i] >= 0) {
      const bool is_q = col[i] < nq;
      const float* w = is_q ? p.qw : p.kw;
      if (w) {
        const int c = is_q ? col[i] : col[i] - nq;
        ldw<VEC>(w + c, wa[i]);
        if (pair[i]) ldw<VEC>(w + c + p.pairs, wb[i]);
      }
    }
  }
  Raw a[KEEP], b[KEEP];
  auto load = [&](int t) {
    const T* row = qkv + t * p.ld;
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
      if (col[i] >= 0) {
        a[i] = *reinterpret_cast<const Raw*>(row + col[i]);
        if (pair[i]) b[i] = *reinterpret_cast<const Raw*>(row + col[i] + p.pairs);
      }
  };
  int t = blockIdx.x, buf = 0;
  if (t < rows) load(t);
  for (; t < rows; t += gridDim.x, buf ^= 1) {
    long long slot = p.slots[t];
    if (slot >= p.num_slots) {
      if (p.status && tid == 0) atomicCAS(p.status, 0, EDL_BAD_INDEX);
      slot = -1;
    }
    if (slot >= 0)
      for (int c = tid * VEC; c < nv; c += blockDim.x * VEC)
        *reinterpret_cast<Raw*>(v_pages + slot * p.ld_vpage + c) =
            *reinterpret_cast<const Raw*>(qkv + t * p.ld + nq + nk + c);
    const float fp = p.pairs ? (float)p.pos[t] : 0.f;
    for (int i = tid; i < p.pairs; i += blockDim.x) cs[buf][i] = turn_of(p, fp, i);
    float va[KEEP][VEC], vb[KEEP][VEC], sq = 0.f, sk = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      if (col[i] < 0) continue;
      ldv<VEC>(reinterpret_cast<const T*>(&a[i]), va[i]);
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < VEC; ++j) s += va[i][j] * va[i][j];
      if (pair[i]) {
        ldv<VEC>(reinterpret_cast<const T*>(&b[i]), vb[i]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) s += vb[i][j] * vb[i][j];
      }
      if (col[i] < nq) sq += s; else sk += s;
    }
    if (t + (int)gridDim.x < rows) load(t + gridDim.x);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) red[buf][warp] = make_float2(sq, sk);
    __syncthreads();
    float2 sums = lane < warps ? red[buf][lane] : make_float2(0.f, 0.f);
    sums.x = warp_sum(sums.x);
    sums.y = warp_sum(sums.y);
    const float rq = p.qw ? 1.f / sqrtf(sums.x / (float)nq + p.eps) : 1.f;
    const float rk = p.kw ? 1.f / sqrtf(sums.y / (float)nk + p.eps) : 1.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
      if (col[i] < 0) continue;
      const bool is_q = col[i] < nq;
      if (!is_q && slot < 0) continue;
      const float r = is_q ? rq : rk;
      T* dst = is_q ? q_out + (long long)t * nq + col[i] : k_pages + slot * p.ld_kpage + (col[i] - nq);
#pragma unroll
      for (int j = 0; j < VEC; ++j) va[i][j] *= r * wa[i][j];
      if (pair[i]) {
        const int c0 = col[i] % p.D;
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
          const float2 g = cs[buf][c0 + j];
          const float x = va[i][j], y = vb[i][j] * (r * wb[i][j]);
          va[i][j] = x * g.x - y * g.y;
          vb[i][j] = y * g.x + x * g.y;
        }
        stv<VEC>(dst + p.pairs, vb[i]);
      }
      stv<VEC>(dst, va[i]);
    }
  }
}

template <typename T, int VEC>
bool launch_rotary_walk(const void* qkv, void* q_out, void* k_pages, void* v_pages, const RotaryPrologueParams& p, int rows,
                        cudaStream_t s) {
  const int units = (p.Hq + p.Hkv) * (p.pairs / VEC + (p.D - 2 * p.pairs) / VEC);
  const int keep = units <= RW_THREADS ? 1 : 2;
  if (units > 2 * RW_THREADS) return false;
  const int threads = ((units + keep - 1) / keep + 31) / 32 * 32;
  const int grid = min(rows, sm_count() * max(1, 1024 / threads));
#define EDL_RW(K) \
  qkv_rotary_walk_kernel<T, VEC, K><<<grid, threads, 0, s>>>((const T*)qkv, (T*)q_out, (T*)k_pages, (T*)v_pages, p, rows)
  if (keep == 1) EDL_RW(1); else EDL_RW(2);
#undef EDL_RW
  return true;
}

// Without norms nothing ties a token's heads together: a CTA takes a few tokens, forms their cosines, and then every warp
// streams one token's pieces (q and k heads, then values).
constexpr int TURN_WARPS = 8;
constexpr int TURN_PAIRS = 2048;      // cosines of a CTA

template <typename T, int VEC>
__global__ void __launch_bounds__(TURN_WARPS * 32)
qkv_turn_kernel(const T* __restrict__ qkv, T* __restrict__ q_out, T* __restrict__ k_pages, T* __restrict__ v_pages,
                const RotaryPrologueParams p, int rows, int tokens, int shift) {
  __shared__ float2 cs[TURN_PAIRS];
  const int t0 = blockIdx.x * tokens, n = min(tokens, rows - t0);
  for (int i = threadIdx.x; i < n * p.pairs; i += TURN_WARPS * 32) {
    const int t = i / p.pairs;
    cs[i] = turn_of(p, (float)p.pos[t0 + t], i - t * p.pairs);
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, split = TURN_WARPS / tokens;    // warps of a token
  const int mine = warp / split, sub = warp - mine * split;
  if (mine >= n) return;
  const int t = t0 + mine;
  const bool inside = p.neighbours && VEC > 1;
  const int turned = (inside ? 2 : 1) * p.pairs / VEC, per = turned + (p.D - 2 * p.pairs) / VEC;
  const int nq = p.Hq * p.D, nk = p.Hkv * p.D, heads = p.Hq + p.Hkv, vunits = p.Hkv * p.Dv / VEC;
  const float2* g = cs + mine * p.pairs;
  const T* row = qkv + t * p.ld;
  long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (p.status && lane == 0) atomicCAS(p.status, 0, EDL_BAD_INDEX);
    slot = -1;
  }
  const int units = slot >= 0 ? heads * per : p.Hq * per;
  T* kdst = k_pages + slot * p.ld_kpage;
#pragma unroll 4
  for (int i = sub * 32 + lane; i < units; i += split * 32) {
    const int h = shift >= 0 ? i >> shift : i / per;
    const T* src = row + h * p.D;
    T* dst = h < p.Hq ? q_out + (long long)t * nq + h * p.D : kdst + (h - p.Hq) * p.D;
    turn_unit<T, VEC>(p, src, dst, h * p.D, nullptr, 1.f, i - h * per, turned, g);
  }
  if (slot >= 0)
#pragma unroll 2
    for (int i = sub * 32 + lane; i < vunits; i += split * 32) {
      float v[VEC];
      ldv<VEC>(row + nq + nk + i * VEC, v);
      finish_values<T, VEC>(p, t, i * VEC, nq + nk + i * VEC, v);
      stv<VEC>(v_pages + slot * p.ld_vpage + i * VEC, v);
    }
}

template <typename T, int VEC>
void launch_turn(const void* qkv, void* q_out, void* k_pages, void* v_pages, const RotaryPrologueParams& p, int rows,
                 cudaStream_t s) {
  int tokens = TURN_WARPS;                // of a CTA: a power of two, fewer when there are few of them
  while (tokens > 1 && (rows < 2 * sm_count() * tokens || tokens * p.pairs > TURN_PAIRS)) tokens >>= 1;
  const int per = ((p.neighbours && VEC > 1 ? 2 : 1) * p.pairs + p.D - 2 * p.pairs) / VEC;
  int shift = -1;
  if ((per & (per - 1)) == 0)
    for (shift = 0; (1 << shift) < per; ++shift) {
    }
  qkv_turn_kernel<T, VEC><<<(rows + tokens - 1) / tokens, TURN_WARPS * 32, 0, s>>>(
      (const T*)qkv, (T*)q_out, (T*)k_pages, (T*)v_pages, p, rows, tokens, shift);
}

// ---- a normed branch joins the stream ----------------------------------------------------------------------------------------
// x <- x + rms_norm(y) * wb * ls, h = rms_norm(x) * w: one CTA per row. NV as above (0: wide rows are read again).
template <typename TO, int VEC, int NV>
__global__ void __launch_bounds__(NT)
branch_norm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ wb,
                   const float* __restrict__ ls, float eps_b, const float* __restrict__ w, float eps, TO* __restrict__ h,
                   int W) {
  __shared__ float2 red[NT / 32];
  constexpr int STEP = NT * VEC, KEEP = NV > 0 ? NV : 1;
  const long long at = (long long)blockIdx.x * W;
  float* xr = x + at;
  const float* yr = y + at;
  float a[KEEP][VEC], s[KEEP][VEC];
  float sum = 0.f;
  // branch rows and stream rows are fetched together, so that the two sums wait for memory once
  auto fetch = [&](int c, float (&ya)[VEC], float (&xa)[VEC]) {
    ldv<VEC>(yr + c, ya);
    ldv<VEC>(xr + c, xa);
#pragma unroll
    for (int j = 0; j < VEC; ++j) sum += ya[j] * ya[j];
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * VEC + k * STEP;
      if (c < W) fetch(c, a[k], s[k]);
    }
  } else {
    for (int c = threadIdx.x * VEC; c < W; c += STEP) fetch(c, a[0], s[0]);
  }
  const float rb = 1.f / sqrtf(block_sum2(sum, 0.f, red).x / (float)W + eps_b);
  sum = 0.f;
  auto join = [&](int c, const float (&ya)[VEC], float (&xa)[VEC]) {
    float wv[VEC], lv[VEC];
    ldv<VEC>(wb + c, wv);
    if (ls) ldv<VEC>(ls + c, lv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      float b = ya[j] * rb * wv[j];
      if (ls) b *= lv[j];
      xa[j] += b;
      sum += xa[j] * xa[j];
    }
    stv<VEC>(xr + c, xa);
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * VEC + k * STEP;
      if (c < W) join(c, a[k], s[k]);
    }
  } else {
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(yr + c, a[0]);
      ldv<VEC>(xr + c, s[0]);
      join(c, a[0], s[0]);         // read back below by the thread that wrote it
    }
  }
  const float rs = 1.f / sqrtf(block_sum2(sum, 0.f, red).x / (float)W + eps);
  auto emit = [&](int c, const float (&xa)[VEC]) {
    float wv[VEC], o[VEC];
    ldv<VEC>(w + c, wv);
#pragma unroll
    for (int j = 0; j < VEC; ++j) o[j] = xa[j] * rs * wv[j];
    stv<VEC>(h + at + c, o);
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int c = threadIdx.x * VEC + k * STEP;
      if (c < W) emit(c, s[k]);
    }
  } else {
    for (int c = threadIdx.x * VEC; c < W; c += STEP) {
      ldv<VEC>(xr + c, s[0]);
      emit(c, s[0]);
    }
  }
}

template <typename TO, int VEC>
void launch_branch_norm(float* x, const float* y, const float* wb, const float* ls, float eps_b, const float* w, float eps,
                        TO* h, int rows, int W, cudaStream_t s) {
  const int nv = (W + NT * VEC - 1) / (NT * VEC);
#define EDL_BN(N) branch_norm_kernel<TO, VEC, N><<<rows, NT, 0, s>>>(x, y, wb, ls, eps_b, w, eps, h, W)
  if (nv <= 1) EDL_BN(1);
  else if (nv <= 2) EDL_BN(2);
  else if (nv <= 4) EDL_BN(4);
  else if (nv <= 8) EDL_BN(8);
  else EDL_BN(0);
#undef EDL_BN
}

// ---- gated units of any size -------------------------------------------------------------------------------------------------
enum { ACT_SILU = 0, ACT_GELU_TANH = 1, ACT_GELU_ERF = 2, ACT_RELU = 3 };

__device__ __forceinline__ float act_of(float z, int act) {
  if (act == ACT_SILU) return z / (1.f + expf(-z));
  if (act == ACT_GELU_TANH) return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  if (act == ACT_GELU_ERF) return 0.5f * z * (1.f + erff(z * 0.7071067811865476f));
  return fmaxf(z, 0.f);
}

// out [T, F] = act(gu[:, :F]) * gu[:, F:]
template <typename T, int VEC>
__global__ void __launch_bounds__(NT)
gated_unit_kernel(const T* __restrict__ gu, long long ld, T* __restrict__ out, int rows, int F, int act) {
  const int per = F / VEC;
  const long long total = (long long)rows * per;
  for (long long i = blockIdx.x * (long long)NT + threadIdx.x; i < total; i += (long long)gridDim.x * NT) {
    const int r = (int)(i / per), c = (int)(i - (long long)r * per) * VEC;
    float g[VEC], u[VEC];
    ldv<VEC>(gu + r * ld + c, g);
    ldv<VEC>(gu + r * ld + F + c, u);
#pragma unroll
    for (int j = 0; j < VEC; ++j) g[j] = act_of(g[j], act) * u[j];
    stv<VEC>(out + (long long)r * F + c, g);
  }
}

// ---- logits ------------------------------------------------------------------------------------------------------------------
template <int VEC>
__global__ void __launch_bounds__(NT) scale_cap_kernel(float* __restrict__ z, long long n_vec, float scale, float cap) {
  const float k = cap > 0.f ? scale / cap : scale;
  for (long long i = blockIdx.x * (long long)NT + threadIdx.x; i < n_vec; i += (long long)gridDim.x * NT) {
    float v[VEC];
    ldv<VEC>(z + i * VEC, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = cap > 0.f ? cap * tanhf(v[j] * k) : v[j] * k;
    stv<VEC>(z + i * VEC, v);
  }
}

int blocks_for(long long work, int per_block, int waves) {
  long long b = (work + per_block - 1) / per_block, cap = (long long)sm_count() * waves;
  return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

template <typename TO, int VEC>
int launch_norm_shift(const float* x, const float* w, const float* mu, float eps, int rows, int W, const int* cu,
                      int nseq, const int* slots, float* state, long long ld_state, float offset, TO* out,
                      cudaStream_t s) {
  const int nv = (W + NT * VEC - 1) / (NT * VEC);
  if (VEC == 4 && nv <= 4 && rows >= 16 * sm_count()) {
    const int per = mu ? 8 : 2;
    const int grid = (rows + per - 1) / per;
#define EDL_NR(N) \
  norm_shift_rows_kernel<TO, N><<<grid, NT, 0, s>>>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset, out, per)
    if (nv <= 1) EDL_NR(1);
    else if (nv <= 2) EDL_NR(2);
    else EDL_NR(4);
#undef EDL_NR
    return check_cuda(cudaGetLastError(), "norm_shift launch");
  }
#define EDL_NS(N) \
  norm_shift_kernel<TO, VEC, N><<<rows, NT, 0, s>>>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset, out)
  if (nv <= 1) EDL_NS(1);
  else if (nv <= 2) EDL_NS(2);
  else if (nv <= 4) EDL_NS(4);
  else if (nv <= 8) EDL_NS(8);
  else EDL_NS(0);
#undef EDL_NS
  return check_cuda(cudaGetLastError(), "norm_shift launch");
}

bool al(const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

}  // namespace
}  // namespace edl

using namespace edl;

// x [rows, W] fp32 = table[ids] * scale; right (may be null): the same rows in the table's type at pitch ld_right.
EDL_HOST_API int edl_embed_stream(const void* table, int f32, const long long* ids, float scale, float* x, void* right,
                                  long long ld_right, int rows, int W, int V, int* status, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = W % 4 == 0 && ld_right % 4 == 0 && al(table, 16) && al(x, 16) && (!right || al(right, 8));
  const int vec = v4 ? 4 : 1;
  const int blocks = blocks_for((long long)rows * (W / vec), 256, 8);
#define EDL_E(T, V_)                                                                                               \
  embed_stream_kernel<T, V_><<<blocks, 256, 0, s>>>((const T*)table, ids, scale, x, (T*)right, ld_right, rows, W, V, status)
  if (f32) {
    if (v4 && (!right || al(right, 16))) EDL_E(float, 4); else EDL_E(float, 1);
  } else {
    if (v4) EDL_E(__nv_bfloat16, 4); else EDL_E(__nv_bfloat16, 1);
  }
#undef EDL_E
  return check_cuda(cudaGetLastError(), "embed_stream launch");
}

// out [rows, :W] at pitch ld_out = x [rows, W] in the operand type.
EDL_HOST_API int edl_cast_rows(const float* x, void* out, int f32, long long ld_out, int rows, int W, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = W % 4 == 0 && ld_out % 4 == 0 && al(x, 16) && al(out, f32 ? 16 : 8);
  const int blocks = blocks_for((long long)rows * (W / (v4 ? 4 : 1)), 256, 8);
#define EDL_C(T, V_) cast_rows_kernel<T, V_><<<blocks, 256, 0, s>>>(x, (T*)out, ld_out, rows, W)
  if (f32) {
    if (v4) EDL_C(float, 4); else EDL_C(float, 1);
  } else {
    if (v4) EDL_C(__nv_bfloat16, 4); else EDL_C(__nv_bfloat16, 1);
  }
#undef EDL_C
  return check_cuda(cudaGetLastError(), "cast_rows launch");
}

// out [rows, W] = rms_norm(x) * (w + offset), blended with the previous row's norm by mu when mu is given. cu [nseq + 1]
// bounds the sequences on the row axis; state [*, ld_state] fp32 holds, per slot, the normalised row before the step's first one
// (null: sequences start here) and is updated to the step's last row.
EDL_HOST_API int edl_norm_shift(const float* x, const float* w, const float* mu, float eps, int rows, int W,
                                const int* cu, int nseq, const int* slots, float* state, long long ld_state, float offset,
                                void* out, int f32, void* stream) {
  if (rows <= 0) return 0;
  if (mu && (!cu || nseq <= 0 || (state && !slots))) {
    set_last_error("edl_norm_shift: a token shift needs sequence bounds, and slots for a state");
    return -1;
  }
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = W % 4 == 0 && ld_state % 4 == 0 && al(x, 16) && al(w, 16) && (!mu || al(mu, 16)) &&
                  (!state || al(state, 16)) && al(out, f32 ? 16 : 8);
  if (f32)
    return v4 ? launch_norm_shift<float, 4>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset, (float*)out, s)
              : launch_norm_shift<float, 1>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset, (float*)out, s);
  return v4 ? launch_norm_shift<__nv_bfloat16, 4>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset,
                                                  (__nv_bfloat16*)out, s)
            : launch_norm_shift<__nv_bfloat16, 1>(x, w, mu, eps, rows, W, cu, nseq, slots, state, ld_state, offset,
                                                  (__nv_bfloat16*)out, s);
}

// o [items, V] fp32 -> rms_norm over V times w.
EDL_HOST_API int edl_head_norm(const float* o, const float* w, float eps, long long items, int V, void* out, int f32,
                               void* stream) {
  if (items <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int blocks = blocks_for(items, NT / 32, 16);
  if (f32) head_norm_kernel<float><<<blocks, NT, 0, s>>>(o, w, eps, items, V, (float*)out);
  else head_norm_kernel<__nv_bfloat16><<<blocks, NT, 0, s>>>(o, w, eps, items, V, (__nv_bfloat16*)out);
  return check_cuda(cudaGetLastError(), "head_norm launch");
}

// y = xielu(z), n elements; act = the two raw parameters (fp32, on the device).
EDL_HOST_API int edl_xielu(const void* z, const float* act, void* y, int f32, long long n, void* stream) {
  if (n <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = n % 4 == 0 && al(z, f32 ? 16 : 8) && al(y, f32 ? 16 : 8);
  const bool v8 = !f32 && n % 8 == 0 && al(z, 16) && al(y, 16);
  const int blocks = blocks_for(n / (v8 ? 8 : v4 ? 4 : 1), 256, 8);
#define EDL_X(T, V_) xielu_kernel<T, V_><<<blocks, 256, 0, s>>>((const T*)z, act, (T*)y, n / V_)
  if (f32) {
    if (v4) EDL_X(float, 4); else EDL_X(float, 1);
  } else {
    if (v8) EDL_X(__nv_bfloat16, 8);
    else if (v4) EDL_X(__nv_bfloat16, 4);
    else EDL_X(__nv_bfloat16, 1);
  }
#undef EDL_X
  return check_cuda(cudaGetLastError(), "xielu launch");
}

EDL_HOST_API int edl_qkv_prologue(const void* qkv, int f32, long long ld, const int* pos, const int* slots,
                                  const float* qw, const float* kw, float eps, float coef, float every, int T, int Hq,
                                  int Hkv, int D, int Dv, void* q_out, void* k_pages, void* v_pages,
                                  long long ld_kpage, long long ld_vpage, long long num_slots, int* status,
                                  void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || Dv <= 0 || !slots || (every > 0.f && !pos)) {
    set_last_error("edl_qkv_prologue: bad arguments (Hq=%d, Hkv=%d, D=%d, Dv=%d)", Hq, Hkv, D, Dv);
    return -1;
  }
  cudaStream_t s = (cudaStream_t)stream;
  const size_t a = f32 ? 16 : 8;
  const bool v4 = D % 4 == 0 && Dv % 4 == 0 && ld % 4 == 0 && ld_kpage % 4 == 0 && ld_vpage % 4 == 0 && al(qkv, a) &&
                  al(q_out, a) && al(k_pages, a) && al(v_pages, a);
  if (v4 && D <= 128 && Dv <= 128 && (long long)T * (Hq + 2 * Hkv) < (1LL << 30)) {
    const int nb = blocks_for((long long)T * ((Hq + 2 * Hkv + 3) / 4), NT / 32, 8);
    if (f32)
      qkv_prologue_small_kernel<float><<<nb, NT, 0, s>>>((const float*)qkv, ld, pos, slots, qw, kw, eps, coef, every, T,
                                                         Hq, Hkv, D, Dv, (float*)q_out, (float*)k_pages,
                                                         (float*)v_pages, ld_kpage, ld_vpage, num_slots, status);
    else
      qkv_prologue_small_kernel<__nv_bfloat16><<<nb, NT, 0, s>>>(
          (const __nv_bfloat16*)qkv, ld, pos, slots, qw, kw, eps, coef, every, T, Hq, Hkv, D, Dv,
          (__nv_bfloat16*)q_out, (__nv_bfloat16*)k_pages, (__nv_bfloat16*)v_pages, ld_kpage, ld_vpage, num_slots,
          status);
    return check_cuda(cudaGetLastError(), "qkv_prologue launch");
  }
  const int blocks = blocks_for((long long)T * (Hq + 2 * Hkv), NT / 32, 8);
#define EDL_P(TT, V_)                                                                                                \
  qkv_prologue_kernel<TT, V_><<<blocks, NT, 0, s>>>((const TT*)qkv, ld, pos, slots, qw, kw, eps, coef, every, T, Hq, \
                                                    Hkv, D, Dv, (TT*)q_out, (TT*)k_pages, (TT*)v_pages, ld_kpage,    \
                                                    ld_vpage, num_slots, status)
  if (f32) {
    if (v4) EDL_P(float, 4); else EDL_P(float, 1);
  } else {
    if (v4) EDL_P(__nv_bfloat16, 4); else EDL_P(__nv_bfloat16, 1);
  }
#undef EDL_P
  return check_cuda(cudaGetLastError(), "qkv_prologue launch");
}

// The prologue for queries and keys that are normed over all heads at once (qw [Hq * D], kw [Hkv * D], null: no norm) and
// rotated, by halves or by neighbours (freq: 2 * pairs floats, leading and trailing parts; pairs = 0: no rotation; mag: factor
// of cosines and sines). bias [Hq * D + Hkv * (D + Dv)] (may be null) is added first; with lam the cached values are
// (1 - *lam) v + *lam v_first, v_first [T, Hkv * Dv] at pitch ld_first.
EDL_HOST_API int edl_qkv_rotary_prologue(const void* qkv, int f32, long long ld, const int* pos, const int* slots,
                                         const float* qw, const float* kw, float eps, const float* freq, int pairs,
                                         int neighbours, float mag, const float* bias, const void* v_first,
                                         long long ld_first, const float* lam, int T, int Hq, int Hkv, int D, int Dv,
                                         void* q_out, void* k_pages, void* v_pages, long long ld_kpage, long long ld_vpage,
                                         long long num_slots, int* status, void* stream) {
  if (T <= 0) return 0;
  if (Hq <= 0 || Hkv <= 0 || D <= 0 || Dv <= 0 || !slots || pairs < 0 || 2 * pairs > D || pairs > RP_MAX_PAIRS ||
      (pairs > 0 && (!pos || !freq)) || (lam && !v_first)) {
    set_last_error("edl_qkv_rotary_prologue: bad arguments (Hq=%d, Hkv=%d, D=%d, Dv=%d, pairs=%d)", Hq, Hkv, D, Dv, pairs);
    return -1;
  }
  const RotaryPrologueParams p{ld,       pos,       slots,  qw,         kw,  eps,  freq,    pairs,    Hq,  Hkv, D, Dv,
                               ld_kpage, ld_vpage, num_slots, status, neighbours, mag, bias, v_first, ld_first, lam};
  cudaStream_t s = (cudaStream_t)stream;
  auto fits = [&](int m, size_t a) {
    return D % m == 0 && (neighbours ? 2 * pairs : pairs) % m == 0 && Dv % m == 0 && ld % m == 0 &&
           (!lam || (ld_first % m == 0 && al(v_first, a))) && ld_kpage % m == 0 && ld_vpage % m == 0 &&
           al(qkv, a) && al(q_out, a) && al(k_pages, a) && al(v_pages, a) && (!qw || al(qw, 16)) && (!kw || al(kw, 16)) &&
           (!bias || al(bias, 16));
  };
#define EDL_RT(TT, V_) launch_turn<TT, V_>(qkv, q_out, k_pages, v_pages, p, T, s)
  if (!qw && !kw) {
    if (f32) {
      if (fits(4, 16)) EDL_RT(float, 4); else EDL_RT(float, 1);
    } else {
      if (fits(8, 16)) EDL_RT(__nv_bfloat16, 8);
      else if (fits(4, 8)) EDL_RT(__nv_bfloat16, 4);
      else EDL_RT(__nv_bfloat16, 1);
    }
    return check_cuda(cudaGetLastError(), "qkv_turn launch");
  }
#undef EDL_RT
  const bool plain = !neighbours && !bias && !lam;
  const bool walked = !plain ? false : f32 ? fits(4, 16) && launch_rotary_walk<float, 4>(qkv, q_out, k_pages, v_pages, p, T, s)
                          : fits(8, 16) && launch_rotary_walk<__nv_bfloat16, 8>(qkv, q_out, k_pages, v_pages, p, T, s);
  if (walked) return check_cuda(cudaGetLastError(), "qkv_rotary_prologue launch");
#define EDL_RP(TT, V_) \
  qkv_rotary_kernel<TT, V_><<<T, NT, 0, s>>>((const TT*)qkv, (TT*)q_out, (TT*)k_pages, (TT*)v_pages, p)
  if (f32) {
    if (fits(4, 16)) EDL_RP(float, 4); else EDL_RP(float, 1);
  } else {
    if (fits(8, 16)) EDL_RP(__nv_bfloat16, 8);
    else if (fits(4, 8)) EDL_RP(__nv_bfloat16, 4);
    else EDL_RP(__nv_bfloat16, 1);
  }
#undef EDL_RP
  return check_cuda(cudaGetLastError(), "qkv_rotary_prologue launch");
}

// x [rows, W] <- x + rms_norm(y) * wb * ls (ls null: 1), h [rows, W] = rms_norm(x) * w in the operand type.
EDL_HOST_API int edl_branch_norm(float* x, const float* y, const float* wb, const float* ls, float eps_b, const float* w,
                                 float eps, void* h, int f32, int rows, int W, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = W % 4 == 0 && al(x, 16) && al(y, 16) && al(wb, 16) && (!ls || al(ls, 16)) && al(w, 16) && al(h, f32 ? 16 : 8);
  if (f32) {
    if (v4) launch_branch_norm<float, 4>(x, y, wb, ls, eps_b, w, eps, (float*)h, rows, W, s);
    else launch_branch_norm<float, 1>(x, y, wb, ls, eps_b, w, eps, (float*)h, rows, W, s);
  } else {
    if (v4) launch_branch_norm<__nv_bfloat16, 4>(x, y, wb, ls, eps_b, w, eps, (__nv_bfloat16*)h, rows, W, s);
    else launch_branch_norm<__nv_bfloat16, 1>(x, y, wb, ls, eps_b, w, eps, (__nv_bfloat16*)h, rows, W, s);
  }
  return check_cuda(cudaGetLastError(), "branch_norm launch");
}

// out [rows, F] = act(gu[:, :F]) * gu[:, F:], gu at pitch ld; act: 0 silu, 1 tanh form of gelu, 2 gelu, 3 relu.
EDL_HOST_API int edl_gated_unit(const void* gu, int f32, long long ld, void* out, int rows, int F, int act, void* stream) {
  if (rows <= 0) return 0;
  if (act < ACT_SILU || act > ACT_RELU) {
    set_last_error("edl_gated_unit: unknown activation %d", act);
    return -1;
  }
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = F % 4 == 0 && ld % 4 == 0 && al(gu, f32 ? 16 : 8) && al(out, f32 ? 16 : 8);
  const int blocks = blocks_for((long long)rows * (F / (v4 ? 4 : 1)), NT, 8);
#define EDL_GU(TT, V_) gated_unit_kernel<TT, V_><<<blocks, NT, 0, s>>>((const TT*)gu, ld, (TT*)out, rows, F, act)
  if (f32) {
    if (v4) EDL_GU(float, 4); else EDL_GU(float, 1);
  } else {
    if (v4) EDL_GU(__nv_bfloat16, 4); else EDL_GU(__nv_bfloat16, 1);
  }
#undef EDL_GU
  return check_cuda(cudaGetLastError(), "gated_unit launch");
}

// z <- cap * tanh(scale * z / cap), n elements in place (cap <= 0: scale * z).
EDL_HOST_API int edl_scale_cap(float* z, long long n, float scale, float cap, void* stream) {
  if (n <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const bool v4 = n % 4 == 0 && al(z, 16);
  const int blocks = blocks_for(n / (v4 ? 4 : 1), NT, 8);
  if (v4) scale_cap_kernel<4><<<blocks, NT, 0, s>>>(z, n / 4, scale, cap);
  else scale_cap_kernel<1><<<blocks, NT, 0, s>>>(z, n, scale, cap);
  return check_cuda(cudaGetLastError(), "scale_cap launch");
}
