// Steps between the products of latent attention and of layers that normalise after the sum, over an fp32 stream.
//
//   * latent prologue: from the packed projection row [queries | latent | rotary key | ...] of a token, the rotary parts of
//     all query heads are rotated where they lie, and the cache row [normalised latent | rotated key] goes to its page;
//   * spans: the pages a step's multi-token portions can still see are numbered densely (a compact page table) and
//     gathered, so that their keys and values can be expanded by one product;
//   * head gate: attention output times sigmoid(gate);
//   * sum and norm: s = alpha x + beta branch, where the branch is a projection's fp32 rows, the weighted sum of expert
//     rows (the combine step of a mixture of experts) or both; the norm of s is the operand of the next product, and x
//     becomes that norm (layers that normalise after the sum) or s itself (layers that normalise before a branch);
//   * exact (erf) GELU.
//
// Compiled without fast-math: these are the parts of such a model that are computed in 32 bits.
#include "common.cuh"

namespace edl {
namespace {

constexpr int NT = 256;

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

// ---- latent prologue -----------------------------------------------------------------------------------------------
constexpr int LP_THREADS = 128;
constexpr int LP_MAX_PAIRS = 256;     // rotated pairs of a head

struct PrologueParams {
  long long ld;              // pitch of a packed row
  const int* pos;
  const int* slots;          // flat page slot of every token (-1: not kept)
  const float* norm_w;       // [L]
  const float* freq;         // [pairs] leading parts of the frequencies, then [pairs] the parts below their last bit
  float eps;
  int H, D, R, L, pairs;     // heads, unrotated and rotary size of a head, latent size, rotated pairs (2 * pairs <= R)
  int halves;                // pair j is (j, j + pairs) of the rotary part instead of its neighbours (2j, 2j + 1)
  long long ld_page, num_slots;
  int* status;
};

// One CTA per token. Angles are p * f with the product's rounding error and the frequency's own carried along as a small
// second rotation, so that they are as exact as 32-bit results can be at any position.
template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_prologue_kernel(T* __restrict__ proj, T* __restrict__ pages, const PrologueParams p) {
  __shared__ float2 cs[LP_MAX_PAIRS];
  __shared__ float red[32];
  const int t = blockIdx.x, tid = threadIdx.x;
  T* row = proj + t * p.ld;
  const T* lat = row + (long long)p.H * (p.D + p.R);
  const float fp = (float)p.pos[t];
  for (int i = tid; i < p.pairs; i += LP_THREADS) {
    const float f = p.freq[i], a = fp * f;
    const float e = fmaf(fp, f, -a) + fp * p.freq[p.pairs + i];
    float s, c;
    sincosf(a, &s, &c);
    const float ce = 1.f - 0.5f * e * e, se = e - e * e * e * (1.f / 6.f);      // e is small: half an ulp of the angle
    cs[i] = make_float2(c * ce - s * se, s * ce + c * se);
  }
  float ss = 0.f;
  for (int c = tid; c < p.L; c += LP_THREADS) {
    const float v = ld1(lat + c);
    ss += v * v;
  }
  ss = block_sum(ss, red);        // its barriers also publish cs
  long long slot = p.slots[t];
  if (slot >= p.num_slots) {
    if (p.status && tid == 0) atomicCAS(p.status, 0, EDL_BAD_INDEX);
    slot = -1;
  }
  if (slot >= 0) {
    T* dst = pages + slot * p.ld_page;
    const float rs = 1.f / sqrtf(ss / (float)p.L + p.eps);
    for (int c = tid; c < p.L; c += LP_THREADS) st1(dst + c, ld1(lat + c) * rs * p.norm_w[c]);
    const T* kr = lat + p.L;
    if (p.halves) {
      for (int i = tid; i < p.R - p.pairs; i += LP_THREADS) {
        if (i < p.pairs) {
          const float u = ld1(kr + i), v = ld1(kr + i + p.pairs);
          const float2 a = cs[i];
          st1(dst + p.L + i, u * a.x - v * a.y);
          st1(dst + p.L + i + p.pairs, v * a.x + u * a.y);
        } else {
          dst[p.L + i + p.pairs] = kr[i + p.pairs];
        }
      }
    }
    for (int i = p.halves ? p.R : tid; i < (p.R + 1) / 2; i += LP_THREADS) {
      if (i < p.pairs) {
        const float u = ld1(kr + 2 * i), v = ld1(kr + 2 * i + 1);
        const float2 a = cs[i];
        st1(dst + p.L + 2 * i, u * a.x - v * a.y);
        st1(dst + p.L + 2 * i + 1, v * a.x + u * a.y);
      } else {
        dst[p.L + 2 * i] = kr[2 * i];
        if (2 * i + 1 < p.R) dst[p.L + 2 * i + 1] = kr[2 * i + 1];
      }
    }
  }
  if (p.halves) {
    // two pairs at a time where the elements come as aligned bf16 pairs
    const bool two = sizeof(T) == 2 && p.pairs % 2 == 0 && (p.D + p.R) % 2 == 0 &&
                     (reinterpret_cast<uintptr_t>(row + p.D) & 3) == 0;
    const int step = two ? 2 : 1, per = p.pairs / step;
    for (int i = tid; i < p.H * per; i += LP_THREADS) {
      const int h = i / per, j = (i - h * per) * step;
      T* q = row + (long long)h * (p.D + p.R) + p.D + j;
      const float2 a = cs[j];
      if constexpr (sizeof(T) == 2) {
        if (two) {
          uint32_t *pu = reinterpret_cast<uint32_t*>(q), *pv = reinterpret_cast<uint32_t*>(q + p.pairs);
          const float2 u = unpack_bf16x2(*pu), v = unpack_bf16x2(*pv), b = cs[j + 1];
          *pu = pack_bf16x2(u.x * a.x - v.x * a.y, u.y * b.x - v.y * b.y);
          *pv = pack_bf16x2(v.x * a.x + u.x * a.y, v.y * b.x + u.y * b.y);
          continue;
        }
      }
      const float u = ld1(q), v = ld1(q + p.pairs);
      st1(q, u * a.x - v * a.y);
      st1(q + p.pairs, v * a.x + u * a.y);
    }
    return;
  }
  const int total = p.H * p.pairs;
  for (int i = tid; i < total; i += LP_THREADS) {
    const int h = i / p.pairs, j = i - h * p.pairs;
    T* q = row + (long long)h * (p.D + p.R) + p.D + 2 * j;
    const float2 a = cs[j];
    if constexpr (sizeof(T) == 2) {
      if ((reinterpret_cast<uintptr_t>(q) & 3) == 0) {
        const float2 uv = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(q));
        *reinterpret_cast<uint32_t*>(q) = pack_bf16x2(uv.x * a.x - uv.y * a.y, uv.y * a.x + uv.x * a.y);
        continue;
      }
    }
    const float u = ld1(q), v = ld1(q + 1);
    st1(q, u * a.x - v * a.y);
    st1(q + 1, v * a.x + u * a.y);
  }
}

// ---- spans -----------------------------------------------------------------------------------------------------------
// One CTA. Sequence b sees pages [first_b, end_b) of its table in this step; they get consecutive compact numbers.
__global__ void __launch_bounds__(NT)
latent_spans_kernel(const int* __restrict__ cu, const int* __restrict__ kv_lens, const int* __restrict__ table,
                    int pt_stride, int B, int window, int page, int cap, int num_pages, int* __restrict__ compact,
                    int* __restrict__ src, int* status) {
  __shared__ int s_base;
  __shared__ int s_sum[NT];
  if (threadIdx.x == 0) s_base = 0;
  __syncthreads();
  for (int b0 = 0; b0 < B; b0 += NT) {
    const int b = b0 + threadIdx.x;
    int first = 0, end = 0;
    if (b < B) {
      const int start = kv_lens[b] - (cu[b + 1] - cu[b]);
      first = window > 0 ? max(0, start - window + 1) / page : 0;
      end = min((kv_lens[b] + page - 1) / page, pt_stride);
      if (cu[b + 1] == cu[b]) end = first;
    }
    s_sum[threadIdx.x] = end - first;
    __syncthreads();
    if (threadIdx.x == 0) {
      int run = s_base;
      for (int i = 0; i < NT; ++i) {
        const int n = s_sum[i];
        s_sum[i] = run;
        run += n;
      }
      s_base = run;
    }
    __syncthreads();
    const int at = s_sum[threadIdx.x];
    if (b < B) {
      for (int j = 0; j < pt_stride; ++j) {
        int v = 0;
        if (j >= first && j < end) {
          v = at + j - first;
          int pg = table[(long long)b * pt_stride + j];
          if (pg < 0 || pg >= num_pages || v >= cap) {
            if (status) atomicCAS(status, 0, EDL_BAD_INDEX);
            pg = 0;
          }
          if (v < cap) src[v] = pg; else v = 0;
        }
        compact[(long long)b * pt_stride + j] = v;
      }
    }
    __syncthreads();
  }
}

template <typename V>
__global__ void gather_pages_kernel(const V* __restrict__ pages, const int* __restrict__ src, V* __restrict__ out,
                                    long long per_page) {
  const V* from = pages + (long long)src[blockIdx.y] * per_page;
  V* to = out + (long long)blockIdx.y * per_page;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < per_page; i += (long long)gridDim.x * blockDim.x)
    to[i] = from[i];
}

// ---- head gate -------------------------------------------------------------------------------------------------------
// out[t, h V + c] = o[t, h, c] * sigmoid(gate[t, h V + c]); o at strides (so_t, so_h).
template <typename T, int VEC>
__global__ void __launch_bounds__(NT)
head_gate_kernel(const T* __restrict__ o, long long so_t, long long so_h, const T* __restrict__ gate, long long ldg,
                 T* __restrict__ out, long long ld_out, int rows, int H, int V) {
  const int per_head = V / VEC, per = H * per_head;
  const long long total = (long long)rows * per;
  for (long long i = blockIdx.x * (long long)NT + threadIdx.x; i < total; i += (long long)gridDim.x * NT) {
    const int t = (int)(i / per), r = (int)(i - (long long)t * per);
    const int h = r / per_head, c = (r - h * per_head) * VEC;
    float a[VEC], g[VEC];
    ldv<VEC>(o + t * so_t + h * so_h + c, a);
    ldv<VEC>(gate + t * ldg + (long long)h * V + c, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      if constexpr (sizeof(T) == 4) a[j] = a[j] / (1.f + expf(-g[j]));
      else a[j] = __fdividef(a[j], 1.f + __expf(-g[j]));
    }
    stv<VEC>(out + t * ld_out + (long long)h * V + c, a);
  }
}

// ---- exact GELU -----------------------------------------------------------------------------------------------------
template <typename T, int VEC>
__global__ void __launch_bounds__(NT) gelu_erf_kernel(const T* __restrict__ z, T* __restrict__ y, long long n_vec) {
  for (long long i = blockIdx.x * (long long)NT + threadIdx.x; i < n_vec; i += (long long)gridDim.x * NT) {
    float v[VEC];
    ldv<VEC>(z + i * VEC, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = 0.5f * v[j] * (1.f + erff(v[j] * 0.70710678118654752f));
    stv<VEC>(y + i * VEC, v);
  }
}

// ---- sum and norm ---------------------------------------------------------------------------------------------------
template <typename TO>
struct PostNormParams {
  float* x;                 // [rows, W] in and out
  const float* y;           // [rows, W] fp32 branch, or null
  const TO* ys;             // expert rows [*, W], or null
  const float* wts;         // [rows, k] weights of the expert rows
  const int* pos;           // [rows, k] their row numbers (< 0: none)
  int k;
  float alpha, beta;
  int keep;                 // x receives the sum, not its norm
  const float* w;           // [W]
  float offset, eps;
  TO* h;                    // [rows, W] operand of the next product
  int rows, W;
};

// NV vectors of VEC elements per thread hold a row; NV = 0: rows wider than that are kept in x between two passes.
template <typename TO, int VEC, int NV>
__global__ void __launch_bounds__(NT) post_norm_kernel(const PostNormParams<TO> p) {
  __shared__ float red[32];
  constexpr int STEP = NT * VEC;
  constexpr int KEEP = NV > 0 ? NV : 1;
  const int r = blockIdx.x;
  float* xr = p.x + (long long)r * p.W;
  float v[KEEP][VEC];
  auto sum_at = [&](int c, float (&a)[VEC]) {
    float m[VEC];
    ldv<VEC>(xr + c, a);
#pragma unroll
    for (int j = 0; j < VEC; ++j) m[j] = 0.f;
    if (p.y) ldv<VEC>(p.y + (long long)r * p.W + c, m);
    if (p.ys) {
      for (int s0 = 0; s0 < p.k; s0 += 4) {       // four rows in flight
        float b[4][VEC], ws[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int at = s0 + u < p.k ? p.pos[(long long)r * p.k + s0 + u] : -1;
          ws[u] = 0.f;
#pragma unroll
          for (int j = 0; j < VEC; ++j) b[u][j] = 0.f;
          if (at >= 0) {
            ws[u] = p.wts[(long long)r * p.k + s0 + u];
            ldv<VEC>(p.ys + (long long)at * p.W + c, b[u]);
          }
        }
#pragma unroll
        for (int u = 0; u < 4; ++u)
#pragma unroll
          for (int j = 0; j < VEC; ++j) m[j] = fmaf(ws[u], b[u][j], m[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) a[j] = fmaf(p.beta, m[j], p.alpha * a[j]);
  };
  float ss = 0.f;
  if constexpr (NV > 0) {
#pragma unroll
    for (int q = 0; q < NV; ++q) {
      const int c = threadIdx.x * VEC + q * STEP;
      if (c < p.W) {
        sum_at(c, v[q]);
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += v[q][j] * v[q][j];
      }
    }
  } else {
    for (int c = threadIdx.x * VEC; c < p.W; c += STEP) {
      sum_at(c, v[0]);
      stv<VEC>(xr + c, v[0]);       // read back below by the thread that wrote it
#pragma unroll
      for (int j = 0; j < VEC; ++j) ss += v[0][j] * v[0][j];
    }
  }
  const float rs = 1.f / sqrtf(block_sum(ss, red) / (float)p.W + p.eps);
  auto emit = [&](int c, float (&a)[VEC]) {
    float wv[VEC];
    ldv<VEC>(p.w + c, wv);
    if (p.keep && NV > 0) stv<VEC>(xr + c, a);
#pragma unroll
    for (int j = 0; j < VEC; ++j) a[j] = a[j] * rs * (wv[j] + p.offset);
    if (!p.keep) stv<VEC>(xr + c, a);
    stv<VEC>(p.h + (long long)r * p.W + c, a);
  };
  if constexpr (NV > 0) {
#pragma unroll
    for (int q = 0; q < NV; ++q) {
      const int c = threadIdx.x * VEC + q * STEP;
      if (c < p.W) emit(c, v[q]);
    }
  } else {
    for (int c = threadIdx.x * VEC; c < p.W; c += STEP) {
      ldv<VEC>(xr + c, v[0]);
      emit(c, v[0]);
    }
  }
}

int blocks_for(long long work, int per_block, int waves) {
  long long b = (work + per_block - 1) / per_block, cap = (long long)sm_count() * waves;
  return (int)(b < 1 ? 1 : (b > cap ? cap : b));
}

bool al(const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; }

template <typename TO, int VEC>
int launch_post_norm(const PostNormParams<TO>& p, cudaStream_t s) {
  const int nv = (p.W + NT * VEC - 1) / (NT * VEC);
#define EDL_PN(N) post_norm_kernel<TO, VEC, N><<<p.rows, NT, 0, s>>>(p)
  if (nv <= 1) EDL_PN(1);
  else if (nv <= 2) EDL_PN(2);
  else if (nv <= 4) EDL_PN(4);
  else if (nv <= 8) EDL_PN(8);
  else EDL_PN(0);
#undef EDL_PN
  return check_cuda(cudaGetLastError(), "post_norm launch");
}

template <typename TO>
int post_norm(float* x, const float* y, const void* ys, const float* wts, const int* pos, int k, float alpha,
              float beta, int keep, const float* w, float offset, float eps, void* h, int rows, int W, cudaStream_t s) {
  PostNormParams<TO> p{x, y, (const TO*)ys, wts, pos, k, alpha, beta, keep, w, offset, eps, (TO*)h, rows, W};
  const size_t a = sizeof(TO) == 4 ? 16 : 8;
  const bool v4 = W % 4 == 0 && al(x, 16) && (!y || al(y, 16)) && (!ys || al(ys, a)) && al(w, 16) && al(h, a);
  return v4 ? launch_post_norm<TO, 4>(p, s) : launch_post_norm<TO, 1>(p, s);
}

}  // namespace
}  // namespace edl

using namespace edl;

// proj [T, ld]: per token H query heads of (D + R), the latent (L), the rotary key (R). The first 2 * pairs of every head's
// R rotary elements are rotated in place (neighbours form a pair, or with `halves` elements j and j + pairs); slots[t] of the page pool [num_slots, ld_page]
// receives [rms_norm(latent) * norm_w | rotated key]. freq: 2 * pairs floats (leading and trailing parts).
EDL_HOST_API int edl_latent_prologue(void* proj, int f32, long long ld, const int* pos, const int* slots,
                                     const float* norm_w, const float* freq, float eps, int T, int H, int D, int R, int L,
                                     int pairs, int halves, void* pages, long long ld_page, long long num_slots, int* status,
                                     void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || D < 0 || R < 0 || L <= 0 || pairs < 0 || 2 * pairs > R || pairs > LP_MAX_PAIRS || !slots || !pos) {
    set_last_error("edl_latent_prologue: bad arguments (H=%d, D=%d, R=%d, L=%d, pairs=%d)", H, D, R, L, pairs);
    return -1;
  }
  PrologueParams p{ld, pos, slots, norm_w, freq, eps, H, D, R, L, pairs, halves, ld_page, num_slots, status};
  cudaStream_t s = (cudaStream_t)stream;
  if (f32) latent_prologue_kernel<float><<<T, LP_THREADS, 0, s>>>((float*)proj, (float*)pages, p);
  else latent_prologue_kernel<__nv_bfloat16><<<T, LP_THREADS, 0, s>>>((__nv_bfloat16*)proj, (__nv_bfloat16*)pages, p);
  return check_cuda(cudaGetLastError(), "latent_prologue launch");
}

// compact [B, pt_stride]: compact page numbers of the pages the step's queries can see (0 elsewhere); src [cap]: their page
// ids. cu [B + 1], kv_lens [B], table [B, pt_stride] as for paged attention; window 0 = none.
EDL_HOST_API int edl_latent_spans(const int* cu, const int* kv_lens, const int* table, int pt_stride, int B, int window,
                                  int page, int cap, int num_pages, int* compact, int* src, int* status, void* stream) {
  if (B <= 0) return 0;
  latent_spans_kernel<<<1, NT, 0, (cudaStream_t)stream>>>(cu, kv_lens, table, pt_stride, B, window, page, cap, num_pages,
                                                          compact, src, status);
  return check_cuda(cudaGetLastError(), "latent_spans launch");
}

// out [n, page_bytes] = pages[src[i]] (page_bytes a multiple of 16).
EDL_HOST_API int edl_gather_pages(const void* pages, const int* src, void* out, int n, long long page_bytes,
                                  void* stream) {
  if (n <= 0) return 0;
  if (page_bytes % 16 || !al(pages, 16) || !al(out, 16) || n > 65535) {
    set_last_error("edl_gather_pages: pages must be 16-byte aligned multiples of 16 bytes, at most 65535 of them");
    return -1;
  }
  const long long per = page_bytes / 16;
  const int bx = (int)((per + 1023) / 1024);
  gather_pages_kernel<uint4><<<dim3(bx, n), NT, 0, (cudaStream_t)stream>>>((const uint4*)pages, src, (uint4*)out, per);
  return check_cuda(cudaGetLastError(), "gather_pages launch");
}

EDL_HOST_API int edl_head_gate(const void* o, int f32, long long so_t, long long so_h, const void* gate, long long ldg,
                               void* out, long long ld_out, int rows, int H, int V, void* stream) {
  if (rows <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int m = f32 ? 4 : 8;
  const bool vec = V % m == 0 && so_t % m == 0 && so_h % m == 0 && ldg % m == 0 && ld_out % m == 0 && al(o, 16) &&
                   al(gate, 16) && al(out, 16);
  const int nb = blocks_for((long long)rows * H * (V / (vec ? m : 1)), NT, 16);
#define EDL_G(T, V_) \
  head_gate_kernel<T, V_><<<nb, NT, 0, s>>>((const T*)o, so_t, so_h, (const T*)gate, ldg, (T*)out, ld_out, rows, H, V)
  if (f32) {
    if (vec) EDL_G(float, 4); else EDL_G(float, 1);
  } else {
    if (vec) EDL_G(__nv_bfloat16, 8); else EDL_G(__nv_bfloat16, 1);
  }
#undef EDL_G
  return check_cuda(cudaGetLastError(), "head_gate launch");
}

EDL_HOST_API int edl_gelu_erf(const void* z, void* y, int f32, long long n, void* stream) {
  if (n <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int m = f32 ? 4 : 8;
  const bool vec = n % m == 0 && al(z, 16) && al(y, 16);
  const int nb = blocks_for(n / (vec ? m : 1), NT, 16);
#define EDL_GE(T, V_) gelu_erf_kernel<T, V_><<<nb, NT, 0, s>>>((const T*)z, (T*)y, n / V_)
  if (f32) {
    if (vec) EDL_GE(float, 4); else EDL_GE(float, 1);
  } else {
    if (vec) EDL_GE(__nv_bfloat16, 8); else EDL_GE(__nv_bfloat16, 1);
  }
#undef EDL_GE
  return check_cuda(cudaGetLastError(), "gelu_erf launch");
}

// x [rows, W] fp32: s = alpha x + beta branch; h (fp32 or bf16) = rms_norm(s) * (w + offset), and x becomes the same (keep =
// 0) or s (keep = 1). The branch is y (fp32 rows), or sum_s wts[r, s] * ys[pos[r, s]] over expert rows in h's type, or both.
EDL_HOST_API int edl_post_norm(float* x, const float* y, const void* ys, const float* wts, const int* pos, int k,
                               float alpha, float beta, int keep, const float* w, float offset, float eps, void* h,
                               int f32, int rows, int W, void* stream) {
  if (rows <= 0) return 0;
  if (ys && (!wts || !pos || k <= 0)) {
    set_last_error("edl_post_norm: expert rows need weights and positions");
    return -1;
  }
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? post_norm<float>(x, y, ys, wts, pos, k, alpha, beta, keep, w, offset, eps, h, rows, W, s)
             : post_norm<__nv_bfloat16>(x, y, ys, wts, pos, k, alpha, beta, keep, w, offset, eps, h, rows, W, s);
}
