// Paged causal attention on the general-purpose cores: any head sizes up to 2048 (query / key) and 1024 (value), bf16 or
// fp32 storage, all arithmetic in fp32. It serves fp32 models (true 32-bit products, which the tensor cores do not have)
// and head sizes outside the tensor-core kernels' tiles.
//
// One CTA per (query token, query head) walks the keys a page at a time: one key per thread for the scores, then one
// value column per thread for the weighted sum, with an online softmax between them (or weights that are sigmoids and need
// no normalisation). The sink logit of a head joins the denominator once at the end. Compiled without fast-math.
#include "common.cuh"

namespace edl {
namespace {

constexpr int ST = 128;      // threads = keys per tile = tokens per page
constexpr int MAX_D = 2048;
constexpr int MAX_VC = 8;    // value columns per thread (Dv <= 1024)

__device__ __forceinline__ float f_of(float v) { return v; }
__device__ __forceinline__ float f_of(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

template <typename T>
__device__ __forceinline__ float dot_row(const T* k, const float* q, int D, bool vec) {
  float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
  if (vec) {
    for (int c = 0; c < D; c += 4) {
      if constexpr (sizeof(T) == 4) {
        const float4 x = *reinterpret_cast<const float4*>(k + c);
        a0 = fmaf(x.x, q[c], a0);
        a1 = fmaf(x.y, q[c + 1], a1);
        a2 = fmaf(x.z, q[c + 2], a2);
        a3 = fmaf(x.w, q[c + 3], a3);
      } else {
        const uint2 x = *reinterpret_cast<const uint2*>(k + c);
        const float2 lo = unpack_bf16x2(x.x), hi = unpack_bf16x2(x.y);
        a0 = fmaf(lo.x, q[c], a0);
        a1 = fmaf(lo.y, q[c + 1], a1);
        a2 = fmaf(hi.x, q[c + 2], a2);
        a3 = fmaf(hi.y, q[c + 3], a3);
      }
    }
  } else {
    for (int c = 0; c < D; ++c) a0 = fmaf(f_of(k[c]), q[c], a0);
  }
  return (a0 + a1) + (a2 + a3);
}

template <typename T>
__global__ void __launch_bounds__(ST)
attn_simt_kernel(const T* __restrict__ q, const T* __restrict__ k_pages, const T* __restrict__ v_pages,
                 T* __restrict__ o, long long ldq, long long ld_kpage, long long ld_vpage, const int* __restrict__ cu,
                 const int* __restrict__ kv_lens, const int* __restrict__ page_table, int pt_stride, int B,
                 long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int window, int keep_first,
                 float softcap, const float* __restrict__ sinks, const float* __restrict__ score_bias,
                 const T* __restrict__ gate, long long ld_gate, float out_scale, long long ldo, bool vec, int* status) {
  __shared__ float sq[MAX_D];
  __shared__ float sp[ST];
  __shared__ float red[32];
  const int t = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int hk = h / (Hq / Hkv);
  int lo = 0, hi = B;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid;
  }
  const int b = lo;
  if (t >= cu[b + 1]) return;                          // rows past the last sequence
  const int qpos = kv_lens[b] - (cu[b + 1] - t);       // the step's tokens end the context
  const int* pt = page_table + (long long)b * pt_stride;
  for (int c = tid; c < D; c += ST) sq[c] = f_of(q[t * ldq + (long long)h * D + c]);
  __syncthreads();
  const int k_lo = window > 0 ? max(0, qpos - window + 1) : 0;
  float m = -INFINITY, l = 0.f;
  float acc[MAX_VC];
#pragma unroll
  for (int i = 0; i < MAX_VC; ++i) acc[i] = 0.f;
  const int first_tile = k_lo / ST, front = window > 0 ? min((keep_first + ST - 1) / ST, first_tile) : 0;
  for (int tile = front > 0 ? 0 : first_tile; tile * ST <= qpos; tile = tile + 1 == front ? first_tile : tile + 1) {
    const long long page = pt[tile];
    if (page < 0 || page >= num_pages) {               // uniform over the CTA
      if (status && tid == 0) atomicCAS(status, 0, EDL_BAD_INDEX);
      continue;
    }
    const int key = tile * ST + tid;
    const bool ok = (key >= k_lo || key < keep_first) && key <= qpos;
    float s = -INFINITY;
    if (ok) s = dot_row(k_pages + (page * ST + tid) * ld_kpage + (long long)hk * D, sq, D, vec) * scale;
    if (ok && softcap > 0.f) s = softcap * tanhf(s / softcap);
    float alpha = 1.f;
    if (score_bias) {                                  // no softmax: weights stand alone
      sp[tid] = ok ? 1.f / (1.f + expf(-(s + score_bias[h]))) : 0.f;
      __syncthreads();
    } else {
      const float m_new = fmaxf(m, block_max(s, red));
      alpha = m == -INFINITY ? 0.f : expf(m - m_new);
      const float p = ok ? expf(s - m_new) : 0.f;
      sp[tid] = p;
      l = l * alpha + block_sum(p, red);               // its barriers also publish sp
      m = m_new;
    }
    const int n = min(ST, qpos - tile * ST + 1);
    const T* vb = v_pages + page * ST * ld_vpage + (long long)hk * Dv;
#pragma unroll
    for (int i = 0; i < MAX_VC; ++i) {
      const int c = tid + i * ST;
      if (c < Dv) {
        float a0 = acc[i] * alpha, a1 = 0.f;
        int j = tile * ST < keep_first ? 0 : max(0, k_lo - tile * ST);      // weights of unseen keys are zero
        for (; j + 1 < n; j += 2) {
          a0 = fmaf(sp[j], f_of(vb[j * ld_vpage + c]), a0);
          a1 = fmaf(sp[j + 1], f_of(vb[(j + 1) * ld_vpage + c]), a1);
        }
        if (j < n) a0 = fmaf(sp[j], f_of(vb[j * ld_vpage + c]), a0);
        acc[i] = a0 + a1;
      }
    }
    __syncthreads();
  }
  float w = 1.f;
  if (sinks) {
    const float m_new = fmaxf(m, sinks[h]);
    w = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * w + expf(sinks[h] - m_new);
  }
  float inv = l > 0.f ? w / l : 0.f;
  if (score_bias) inv = out_scale / (gate ? 1.f + expf(-f_of(gate[t * ld_gate + h])) : 1.f);
#pragma unroll
  for (int i = 0; i < MAX_VC; ++i) {
    const int c = tid + i * ST;
    if (c < Dv) put(o + t * ldo + (long long)h * Dv + c, acc[i] * inv);
  }
}

template <typename T>
int launch_simt(const void* q, const void* k, const void* v, void* o, long long ldq, long long ldk, long long ldv,
                const int* cu, const int* kv_lens, const int* pt, int pt_stride, int B, int T_rows,
                long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int window, int keep_first, float softcap,
                const float* sinks, const float* score_bias, const void* gate, long long ld_gate, float out_scale,
                long long ldo, int* status, cudaStream_t s) {
  const bool vec = D % 4 == 0 && ldk % 4 == 0 && (reinterpret_cast<uintptr_t>(k) & 15) == 0;
  attn_simt_kernel<T><<<dim3(T_rows, Hq), ST, 0, s>>>((const T*)q, (const T*)k, (const T*)v, (T*)o, ldq, ldk, ldv, cu,
                                                      kv_lens, pt, pt_stride, B, num_pages, Hq, Hkv, D, Dv, scale,
                                                      window, keep_first, softcap, sinks, score_bias, (const T*)gate,
                                                      ld_gate, out_scale, ldo, vec, status);
  return check_cuda(cudaGetLastError(), "attn_simt launch");
}

}  // namespace
}  // namespace edl

// q [T, ldq] (head h at columns h * D), key / value pages [num_pages * 128, ld] with the heads packed in a row,
// o [T, ldo] (head h at columns h * Dv); cu [B + 1], kv_lens [B], page_table [B, pt_stride] as in edl_attn_paged; f32: storage
// type; softcap > 0: scores become softcap * tanh(score / softcap); keep_first: keys that stay visible under a window.
// score_bias [Hq] (may be null): no softmax, weights are sigmoid(score + bias), the output is multiplied by out_scale and, with a
// gate [T, ld_gate] in the storage type, by sigmoid(gate[t][h]).
EDL_HOST_API int edl_attn_simt(const void* q, const void* k_pages, const void* v_pages, void* o, int f32,
                               long long ldq, long long ld_kpage, long long ld_vpage, long long ldo, const int* cu,
                               const int* kv_lens, const int* page_table, int pt_stride, int B, int T,
                               long long num_pages, int Hq, int Hkv, int D, int Dv, float scale, int window, int keep_first,
                               float softcap, const float* sinks, const float* score_bias, const void* gate,
                               long long ld_gate, float out_scale, int* status, void* stream) {
  using namespace edl;
  if (B <= 0 || T <= 0) return 0;
  if (D < 1 || D > MAX_D || Dv < 1 || Dv > MAX_VC * ST || Hkv < 1 || Hq % Hkv || Hq > 65535) {
    set_last_error("edl_attn_simt: unsupported head layout (D=%d, Dv=%d, Hq=%d, Hkv=%d)", D, Dv, Hq, Hkv);
    return -1;
  }
  cudaStream_t s = (cudaStream_t)stream;
  return f32 ? launch_simt<float>(q, k_pages, v_pages, o, ldq, ld_kpage, ld_vpage, cu, kv_lens, page_table, pt_stride,
                                  B, T, num_pages, Hq, Hkv, D, Dv, scale, window, keep_first, softcap, sinks, score_bias,
                                  gate, ld_gate, out_scale, ldo, status, s)
             : launch_simt<__nv_bfloat16>(q, k_pages, v_pages, o, ldq, ld_kpage, ld_vpage, cu, kv_lens, page_table,
                                          pt_stride, B, T, num_pages, Hq, Hkv, D, Dv, scale, window, keep_first, softcap,
                                          sinks, score_bias, gate, ld_gate, out_scale, ldo, status, s);
}
