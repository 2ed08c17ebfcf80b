// Routing and expert products of a mixture of experts in inference, around the grouped tcgen05 products of gemm.cu.
//
//   * route, from the router's fp32 logits: either sigmoid scores, choice by score + correction, weights = the chosen
//     scores over their sum; or choice by logit, weights = the softmax over the chosen logits. For the few tokens of a decode step the same launch also buckets the (token, choice) pairs by expert
//     (the tables that edl_moe_route builds in several launches);
//   * gated unit over used rows: silu(g) u, or clamped: g' sigmoid(alpha g') (u' + 1) with g' = min(g, limit), u' =
//     clamp(u, +-limit);
//   * grouped product on the general-purpose cores for models in 32 bits and sizes outside the tensor-core tiles.
//
// Compiled without fast-math.
#include "common.cuh"

namespace edl {
namespace {

constexpr int SEG = 128;          // rows of a segment's tiles
constexpr int MAX_E = 1024;
constexpr int MAX_TOP = 32;
constexpr int SMALL_PAIRS = 4096; // (token, choice) pairs of the one-launch form
constexpr int SMALL_THREADS = 512;

__device__ __forceinline__ float f_of(float v) { return v; }
__device__ __forceinline__ float f_of(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// One warp routes one token over at most 32 * NE experts. Lane s < top returns the s-th choice and its weight.
template <int NE>
__device__ __forceinline__ void route_token(const float* __restrict__ logits, const float* __restrict__ corr,
                                            bool sigmoid, int E, int top, int lane, int& mine, float& weight) {
  float score[NE], choice[NE];
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    const int e = i * 32 + lane;
    score[i] = e < E ? (sigmoid ? 1.f / (1.f + expf(-logits[e])) : logits[e]) : 0.f;
    choice[i] = e < E ? score[i] + (corr ? corr[e] : 0.f) : -INFINITY;
  }
  mine = 0;
  float got = 0.f;
  for (int s = 0; s < top; ++s) {
    float bv = -INFINITY, bs = 0.f;
    int be = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      if (choice[i] > bv) {
        bv = choice[i];
        be = i * 32 + lane;
        bs = score[i];
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o), os = __shfl_xor_sync(0xffffffffu, bs, o);
      const int oe = __shfl_xor_sync(0xffffffffu, be, o);
      if (ov > bv || (ov == bv && oe < be)) {
        bv = ov;
        be = oe;
        bs = os;
      }
    }
    if (be >= E) be = s;          // only with non-finite logits: keep the index in range
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (i * 32 + lane == be) choice[i] = -INFINITY;
    if (lane == s) {
      mine = be;
      got = bs;
    }
  }
  if (!sigmoid) {                 // lane 0 has the largest logit
    const float top_logit = __shfl_sync(0xffffffffu, got, 0);
    got = lane < top ? expf(got - top_logit) : 0.f;
  }
  weight = got / (warp_sum(got) + 1e-20f);
}

template <int NE>
__global__ void __launch_bounds__(256)
route_kernel(const float* __restrict__ logits, const float* __restrict__ corr, bool sigmoid, int T, int E, int top,
             long long* __restrict__ idx, float* __restrict__ wts) {
  const int lane = threadIdx.x & 31;
  for (int t = blockIdx.x * 8 + (threadIdx.x >> 5); t < T; t += gridDim.x * 8) {
    int e;
    float w;
    route_token<NE>(logits + (long long)t * E, corr, sigmoid, E, top, lane, e, w);
    if (lane < top) {
      idx[(long long)t * top + lane] = e;
      wts[(long long)t * top + lane] = w;
    }
  }
}

// One CTA: routing and the bucket tables of a small step.
template <int NE>
__global__ void __launch_bounds__(SMALL_THREADS)
route_small_kernel(const float* __restrict__ logits, const float* __restrict__ corr, bool sigmoid, int T, int E, int top,
                   float* __restrict__ wts, int* __restrict__ tile_expert, int max_tiles, int* __restrict__ meta,
                   int* __restrict__ slot_pos, int* __restrict__ row_token) {
  __shared__ int count[MAX_E], offset[MAX_E + 1];
  __shared__ short expert_of[SMALL_PAIRS], rank_of[SMALL_PAIRS];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  for (int e = threadIdx.x; e < E; e += SMALL_THREADS) count[e] = 0;
  __syncthreads();
  for (int t = warp; t < T; t += SMALL_THREADS / 32) {
    int e;
    float w;
    route_token<NE>(logits + (long long)t * E, corr, sigmoid, E, top, lane, e, w);
    if (lane < top) {
      const int i = t * top + lane;
      wts[i] = w;
      expert_of[i] = (short)e;
      rank_of[i] = (short)atomicAdd(&count[e], 1);
    }
  }
  __syncthreads();
  if (warp == 0) {                // rows of the experts, padded to whole tiles, one after the other
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + lane;
      const int n = e < E ? (count[e] + SEG - 1) / SEG * SEG : 0;
      int up = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, up, o);
        if (lane >= o) up += v;
      }
      if (e < E) offset[e] = base + up - n;
      base += __shfl_sync(0xffffffffu, up, 31);
    }
    if (lane == 0) {
      offset[E] = base;
      meta[0] = base / SEG;
      meta[1] = base;
    }
  }
  __syncthreads();
  for (int e = warp; e < E; e += SMALL_THREADS / 32) {
    const int lo = offset[e], hi = offset[e + 1];
    for (int t = lo / SEG + lane; t < hi / SEG && t < max_tiles; t += 32) tile_expert[t] = e;
    for (int r = lo + count[e] + lane; r < hi; r += 32) row_token[r] = -1;
  }
  for (int i = threadIdx.x; i < T * top; i += SMALL_THREADS) {
    const int r = offset[expert_of[i]] + rank_of[i];
    slot_pos[i] = r;
    row_token[r] = i / top;
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
glu_kernel(const T* __restrict__ gu, const int* __restrict__ row_token, const int* __restrict__ meta,
           T* __restrict__ out, int F, long long rows, float limit, float alpha) {
  const int per = F / VEC;
  const bool clamped = limit > 0.f;
  const float k = clamped ? alpha : 1.f;
  const long long total = (meta ? (long long)meta[1] : rows) * per;
  for (long long i = blockIdx.x * 256LL + threadIdx.x; i < total; i += gridDim.x * 256LL) {
    const long long r = i / per;
    if (row_token && row_token[r] < 0) continue;
    const int c = (int)(i - r * per) * VEC;
    const T* gp = gu + r * 2 * F + c;
    alignas(16) T g_[VEC], u_[VEC], o_[VEC];
    if constexpr (VEC * sizeof(T) == 16) {
      *reinterpret_cast<uint4*>(g_) = *reinterpret_cast<const uint4*>(gp);
      *reinterpret_cast<uint4*>(u_) = *reinterpret_cast<const uint4*>(gp + F);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) {
        g_[j] = gp[j];
        u_[j] = gp[F + j];
      }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
      float g = f_of(g_[j]), u = f_of(u_[j]), s;
      if (clamped) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit) + 1.f;
      }
      if constexpr (sizeof(T) == 4) s = g / (1.f + expf(-k * g));
      else s = __fdividef(g, 1.f + __expf(-k * g));
      put(&o_[j], s * u);
    }
    T* dst = out + r * F + c;
    if constexpr (VEC * sizeof(T) == 16) {
      *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(o_);
    } else {
#pragma unroll
      for (int j = 0; j < VEC; ++j) dst[j] = o_[j];
    }
  }
}

// out[r, n] = A[row(r), :] . W[e(r)][n, :] for the rows of the segment tables; row(r) = row_token[r] when GATHER (padding
// rows give zeros), else r. 64 x 64 tiles, fp32 arithmetic.
constexpr int GT = 64, GK = 16;
template <typename T, bool GATHER>
__global__ void __launch_bounds__(256)
grouped_simt_kernel(const T* __restrict__ a, long long lda, const int* __restrict__ row_token, const T* __restrict__ w,
                    const int* __restrict__ tile_expert, const int* __restrict__ meta, T* __restrict__ out, int N, int K) {
  const int r0 = blockIdx.y * GT, n0 = blockIdx.x * GT;
  if (r0 >= meta[1]) return;
  __shared__ float sa[GK][GT + 1], sb[GK][GT + 1];
  __shared__ long long src[GT];
  const int tid = threadIdx.x;
  if (tid < GT) src[tid] = GATHER ? row_token[r0 + tid] : (row_token[r0 + tid] < 0 ? -1 : r0 + tid);
  __syncthreads();
  const T* we = w + (long long)tile_expert[r0 / SEG] * N * K;
  const int ty = tid >> 4, tx = tid & 15;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += GK) {
#pragma unroll
    for (int q = 0; q < GT * GK / 256; ++q) {
      const int i = tid + q * 256, r = i / GK, c = i % GK, k = k0 + c;
      sa[c][r] = src[r] >= 0 && k < K ? f_of(a[src[r] * lda + k]) : 0.f;
      sb[c][r] = n0 + r < N && k < K ? f_of(we[(long long)(n0 + r) * K + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < GK; ++c) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        x[i] = sa[c][ty + 16 * i];
        y[i] = sb[c][tx + 16 * i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = r0 + ty + 16 * i, n = n0 + tx + 16 * j;
      if (n < N) put(out + (long long)r * N + n, acc[i][j]);
    }
}

}  // namespace
}  // namespace edl

using namespace edl;

#define EDL_BY_EXPERTS(E, CALL)  \
  do {                           \
    if ((E) <= 32) { CALL(1); }       \
    else if ((E) <= 64) { CALL(2); }  \
    else if ((E) <= 128) { CALL(4); } \
    else if ((E) <= 256) { CALL(8); } \
    else { CALL(32); }                \
  } while (0)

static int check_route(const char* who, int E, int top) {
  if (E < 1 || E > MAX_E || top < 1 || top > MAX_TOP || top > E) {
    set_last_error("%s: 1 to %d experts and 1 to %d choices, got %d and %d", who, MAX_E, MAX_TOP, E, top);
    return -1;
  }
  return 0;
}

// logits [T, E] fp32; corr [E] fp32 or null -> idx [T, top] (best first), wts [T, top]. sigmoid: see the top of the file.
EDL_HOST_API int edl_moe_logit_route(const float* logits, const float* corr, int sigmoid, int T, int E, int top,
                                     long long* idx, float* wts, void* stream) {
  if (T <= 0) return 0;
  if (check_route("edl_moe_logit_route", E, top)) return -1;
  const int cap = 8 * sm_count(), nb = (T + 7) / 8 < cap ? (T + 7) / 8 : cap;
#define EDL_R(NE) route_kernel<NE><<<nb, 256, 0, (cudaStream_t)stream>>>(logits, corr, sigmoid != 0, T, E, top, idx, wts)
  EDL_BY_EXPERTS(E, EDL_R);
#undef EDL_R
  return check_cuda(cudaGetLastError(), "moe_logit_route launch");
}

// Routing plus the bucket tables (tile_expert [max_tiles], meta [2], slot_pos [T * top], row_token [max_tiles * 128]; the
// layout of edl_moe_route) in one launch; T * top <= 4096.
EDL_HOST_API int edl_moe_logit_route_small(const float* logits, const float* corr, int sigmoid, int T, int E, int top,
                                           float* wts, int* tile_expert, int max_tiles, int* meta, int* slot_pos,
                                           int* row_token, void* stream) {
  if (T <= 0) return 0;
  if (check_route("edl_moe_logit_route_small", E, top)) return -1;
  if ((long long)T * top > SMALL_PAIRS || max_tiles < (T * top + SEG - 1) / SEG + (E < T * top ? E : T * top)) {
    set_last_error("edl_moe_logit_route_small: at most %d pairs, and tables for every expert's ragged tile", SMALL_PAIRS);
    return -1;
  }
#define EDL_R(NE)                                                                                                  \
  route_small_kernel<NE><<<1, SMALL_THREADS, 0, (cudaStream_t)stream>>>(logits, corr, sigmoid != 0, T, E, top, wts, \
                                                                        tile_expert, max_tiles, meta, slot_pos, row_token)
  EDL_BY_EXPERTS(E, EDL_R);
#undef EDL_R
  return check_cuda(cudaGetLastError(), "moe_logit_route_small launch");
}

// gu [max_rows, 2F] (gate | up) -> out [max_rows, F], rows in use only (without tables: all rows). limit > 0: clamped unit.
EDL_HOST_API int edl_moe_glu(const void* gu, int f32, const int* row_token, const int* meta, void* out, int F,
                             long long max_rows, float limit, float alpha, void* stream) {
  if (max_rows <= 0 || F <= 0) return 0;
  cudaStream_t s = (cudaStream_t)stream;
  const int m = f32 ? 4 : 8;
  const bool vec = F % m == 0 && ((reinterpret_cast<uintptr_t>(gu) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const long long work = (max_rows * (F / (vec ? m : 1)) + 255) / 256;
  const int cap = 16 * sm_count(), nb = (int)(work < cap ? work : cap);
#define EDL_C(T, V) \
  glu_kernel<T, V><<<nb, 256, 0, s>>>((const T*)gu, row_token, meta, (T*)out, F, max_rows, limit, alpha)
  if (f32) {
    if (vec) EDL_C(float, 4); else EDL_C(float, 1);
  } else {
    if (vec) EDL_C(__nv_bfloat16, 8); else EDL_C(__nv_bfloat16, 1);
  }
#undef EDL_C
  return check_cuda(cudaGetLastError(), "moe_glu launch");
}

// out [max_rows, N] = rows of a times W[e]^T, W [E, N, K]; gather != 0: row r reads a[row_token[r]].
EDL_HOST_API int edl_moe_grouped_simt(const void* a, int f32, long long lda, const int* row_token, int gather,
                                      const void* w, const int* tile_expert, const int* meta, void* out, int max_rows,
                                      int N, int K, void* stream) {
  if (max_rows <= 0 || N <= 0 || K <= 0) return 0;
  if (max_rows % SEG || max_rows / GT > 65535) {
    set_last_error("edl_moe_grouped_simt: max_rows must be a multiple of 128 below 4 million, got %d", max_rows);
    return -1;
  }
  const dim3 grid((N + GT - 1) / GT, max_rows / GT);
  cudaStream_t s = (cudaStream_t)stream;
#define EDL_GS(T, G) \
  grouped_simt_kernel<T, G><<<grid, 256, 0, s>>>((const T*)a, lda, row_token, (const T*)w, tile_expert, meta, (T*)out, N, K)
  if (f32) {
    if (gather) EDL_GS(float, true); else EDL_GS(float, false);
  } else {
    if (gather) EDL_GS(__nv_bfloat16, true); else EDL_GS(__nv_bfloat16, false);
  }
#undef EDL_GS
  return check_cuda(cudaGetLastError(), "moe_grouped_simt launch");
}
