// Shared device/host helpers for the sm_100a kernel library.
//
// Everything here is a thin wrapper over one PTX instruction (mbarrier, TMA,
// tcgen05) or a small host utility (tensor-map encode, error reporting).
// Every wait on an mbarrier is bounded: after `EDL_SPIN_LIMIT_CYCLES` clock
// cycles the waiter records a code in the kernel's status word and gives up,
// so a broken pipeline ends the kernel instead of hanging the GPU.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#ifndef EDL_SPIN_LIMIT_CYCLES
#define EDL_SPIN_LIMIT_CYCLES (3000000000LL)  // ~1.5-2.3 s at B200 clocks
#endif

// Status-word codes written by kernels whose waits ran out.
enum EdlStatus : int {
  EDL_OK = 0,
  EDL_TIMEOUT_PRODUCER = 1,
  EDL_TIMEOUT_MMA = 2,
  EDL_TIMEOUT_EPILOGUE = 3,
  EDL_TIMEOUT_PEER_FLAG = 4,
  EDL_TIMEOUT_SOFTMAX = 5,
  EDL_BAD_INDEX = 6,
};

#define EDL_HOST_API extern "C" __attribute__((visibility("default")))

namespace edl {

// ----------------------------------------------------------------------------
// host side
// ----------------------------------------------------------------------------
void set_last_error(const char* fmt, ...);
int check_cuda(cudaError_t e, const char* what);

// Encodes a 2-D tiled tensor map over a row-major matrix of 16-bit elements:
// `rows` x `cols`, leading dimension `ld` elements, box = box_rows x box_cols,
// 128-byte swizzle (box_cols * 2 bytes must equal 128), zero fill out of range.
// Returns 0 on success.
int make_tmap_2d_16b(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                     uint32_t box_rows, uint32_t box_cols);
// Same, but with an explicit swizzle mode (0 none, 1 32B, 2 64B, 3 128B) and
// element size in bytes (2 or 4).
int make_tmap_2d(CUtensorMap* map, const void* base, uint64_t rows, uint64_t cols, uint64_t ld,
                 uint32_t box_rows, uint32_t box_cols, int elem_bytes, int swizzle);
// 3-D map: dims (d0 innermost, d1, d2) with strides in elements for d1 and d2.
int make_tmap_3d_16b(CUtensorMap* map, const void* base, uint64_t d0, uint64_t d1, uint64_t d2,
                     uint64_t stride1, uint64_t stride2, uint32_t box0, uint32_t box1, uint32_t box2,
                     int swizzle);

int sm_count();

// ----------------------------------------------------------------------------
// device side
// ----------------------------------------------------------------------------
#ifdef __CUDACC__

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}

__device__ __forceinline__ void mbar_init(uint32_t bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count) : "memory");
}
__device__ __forceinline__ void fence_mbar_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}
__device__ __forceinline__ void mbar_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ uint32_t mbar_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(bar), "r"(parity)
      : "memory");
  return ok;
}

// Bounded wait. `abort_flag` is a shared-memory word that any role sets when it
// gives up, so the other roles leave their loops quickly. Returns true when the
// barrier phase completed, false when the wait was abandoned.
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int* abort_flag,
                                          int* status, int code) {
  if (mbar_try_wait(bar, parity)) return true;
  long long t0 = clock64();
  uint32_t it = 0;
  while (true) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((++it & 0x3ff) == 0) {
      if (*abort_flag) return false;
      if (clock64() - t0 > EDL_SPIN_LIMIT_CYCLES) {
        *abort_flag = 1;
        if (status) atomicCAS(status, 0, code);
        return false;
      }
    }
  }
}

// TMA tiled loads. Every load in this library targets the issuing CTA only.
__device__ __forceinline__ void tma_load_2d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y,
                                            int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y), "r"(z)
      : "memory");
}
__device__ __forceinline__ void tma_store_2d(const CUtensorMap* map, uint32_t src, int x, int y) {
  asm volatile("cp.async.bulk.tensor.2d.global.shared::cta.bulk_group [%0, {%2, %3}], [%1];" ::"l"(map), "r"(src),
               "r"(x), "r"(y)
               : "memory");
}
__device__ __forceinline__ void tma_store_commit() { asm volatile("cp.async.bulk.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void tma_store_wait_read() {
  asm volatile("cp.async.bulk.wait_group.read %0;" ::"n"(N) : "memory");
}
template <int N>
__device__ __forceinline__ void tma_store_wait() {
  asm volatile("cp.async.bulk.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void prefetch_tmap(const CUtensorMap* map) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(map) : "memory");
}

// ---- tcgen05 / tensor memory ------------------------------------------------
__device__ __forceinline__ void tmem_alloc(uint32_t smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_dst), "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
// True in exactly one lane of a fully converged warp. A role whose warp stays converged and lets the elected lane
// issue (instead of branching to lane 0 for the whole role) keeps its operand arithmetic on the uniform datapath.
__device__ __forceinline__ bool elect_one() {
  uint32_t pred;
  asm volatile("{\n\t.reg .pred P;\n\telect.sync _|P, 0xffffffff;\n\tselp.u32 %0, 1, 0, P;\n\t}" : "=r"(pred));
  return pred != 0;
}
__device__ __forceinline__ void tc_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void tc_wait_ld() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ void tc_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// D[tmem] (+)= A[smem desc] * B[smem desc]; bf16/f16 inputs, one CTA.
__device__ __forceinline__ void umma_f16_ss(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// D[tmem] (+)= A[tmem] * B[smem desc].
__device__ __forceinline__ void umma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t bdesc, uint32_t idesc,
                                            uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// ---- CTA pairs (cta_group::2): two CTAs of a cluster issue one MMA over both SMs' shared and tensor memory ----
__device__ __forceinline__ uint32_t cluster_ctarank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
// Address of the same shared-memory location in CTA `rank` of this cluster (shared::cluster window).
__device__ __forceinline__ uint32_t mapa_shared(uint32_t addr, uint32_t rank) {
  uint32_t r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
  return r;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// Arrive on an mbarrier that may live in the peer CTA (address from mapa_shared).
__device__ __forceinline__ void mbar_arrive_cluster(uint32_t bar) {
  asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(bar) : "memory");
}
// TMA tile load issued by one CTA of a pair into its own shared memory; the completion bytes go to `bar`, which
// may be the pair leader's barrier. No multicast: each CTA fetches its own tile.
__device__ __forceinline__ void tma_load_2d_pair(uint32_t dst, const CUtensorMap* map, uint32_t bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.cta_group::2.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(dst), "l"(map), "r"(bar), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tmem_alloc_pair(uint32_t smem_dst, uint32_t ncols) {
  asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_dst), "r"(ncols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish_pair() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc_pair(uint32_t taddr, uint32_t ncols) {
  asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(ncols) : "memory");
}
// Arrives on the barrier at this shared-memory offset in every CTA of `cta_mask` once all MMAs issued so far by
// this thread have completed (the arrival is multicast; no data is).
__device__ __forceinline__ void tc_commit_pair(uint32_t bar, uint16_t cta_mask) {
  asm volatile("tcgen05.commit.cta_group::2.mbarrier::arrive::one.shared::cluster.multicast::cluster.b64 [%0], %1;"
               ::"r"(bar), "h"(cta_mask)
               : "memory");
}
// D[tmem of both CTAs] (+)= A * B with M = 256 split over the pair; issued by one thread of the leader CTA.
__device__ __forceinline__ void umma_f16_ss_pair(uint32_t d_tmem, uint64_t adesc, uint64_t bdesc, uint32_t idesc,
                                                 uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::2.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// Instruction descriptor for kind::f16 with bf16 A/B and fp32 D.
// a_mn / b_mn: 1 when the operand's contiguous dimension is M (resp. N), 0 when
// it is K.
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int M, int N, int a_mn, int b_mn) {
  return (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(a_mn) << 15) | (uint32_t(b_mn) << 16) |
         (uint32_t(N >> 3) << 17) | (uint32_t(M >> 4) << 24);
}

// Shared-memory matrix descriptor, 128-byte swizzle, descriptor version 1.
// lbo/sbo in bytes. For K-major tiles (rows of 128 bytes) sbo = 1024 and lbo is
// ignored; for MN-major tiles made of [k-rows x 128-byte] boxes sbo = 1024
// (eight k-rows) and lbo = bytes between consecutive 64-element MN chunks.
__device__ __forceinline__ uint64_t umma_smem_desc_sw128(uint32_t saddr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= uint64_t((saddr & 0x3FFFF) >> 4);
  d |= uint64_t((lbo >> 4) & 0x3FFF) << 16;
  d |= uint64_t((sbo >> 4) & 0x3FFF) << 32;
  d |= uint64_t(1) << 46;  // version
  d |= uint64_t(2) << 61;  // SWIZZLE_128B
  return d;
}

// 32 lanes x 32 consecutive fp32 columns: thread i of the warp gets lane
// (quadrant*32 + i), registers j = column j.
__device__ __forceinline__ void tmem_ld_32x32b_x32(uint32_t taddr, uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, "
      "%16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31}, [%32];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]),
        "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]),
        "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_ld_32x32b_x16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_st_32x32b_x32(uint32_t taddr, const uint32_t (&r)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]),
        "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]),
        "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
      : "memory");
}

__device__ __forceinline__ uint32_t pack_bf16x2(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ float2 unpack_bf16x2(uint32_t u) {
  __nv_bfloat162 v = *reinterpret_cast<__nv_bfloat162*>(&u);
  return __bfloat1622float2(v);
}

// ---- packed fp32 arithmetic and a software exp2 for the softmax loops ----------------------------------------
__device__ __forceinline__ float fmax3(float a, float b, float c) {
  float m;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(m) : "f"(a), "f"(b), "f"(c));
  return m;
}
// (d0, d1) = (a0, a1) * (b0, b1) + (c0, c1) as one packed instruction.
__device__ __forceinline__ void fma2(float& d0, float& d1, float a0, float a1, float b0, float b1, float c0,
                                     float c1) {
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\tmov.b64 rc, {%6, %7};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d0), "=f"(d1)
      : "f"(a0), "f"(a1), "f"(b0), "f"(b1), "f"(c0), "f"(c1));
}
__device__ __forceinline__ void add2(float& d0, float& d1, float a0, float a1) {
  asm("{\n\t.reg .b64 ra, rd;\n\t"
      "mov.b64 rd, {%0, %1};\n\tmov.b64 ra, {%2, %3};\n\t"
      "add.rn.f32x2 rd, rd, ra;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "+f"(d0), "+f"(d1)
      : "f"(a0), "f"(a1));
}
__device__ __forceinline__ void mul2(float& d0, float& d1, float a0, float a1, float b0, float b1) {
  asm("{\n\t.reg .b64 ra, rb, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\t"
      "mul.rn.f32x2 rd, ra, rb;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d0), "=f"(d1)
      : "f"(a0), "f"(a1), "f"(b0), "f"(b1));
}
// 2^x on the FMA and integer pipes (no MUFU): round x to the nearest integer n with the 1.5 * 2^23 trick, a cubic
// for 2^f on f = x - n in [-0.5, 0.5] (relative error 1.0e-4, well under bf16 rounding), then n added to the
// exponent field. Used for a share of the softmax exponentials, whose MUFU throughput (16 per clock and SM)
// otherwise bounds attention. x <= -126 (masked scores included) gives a value below 1e-37.
__device__ __forceinline__ float exp2_poly(float x) {
  x = fmaxf(x, -126.f);
  const float t = x + 12582912.f;
  const float f = x - (t - 12582912.f);
  float p = fmaf(0.05592204f, f, 0.24264008f);
  p = fmaf(p, f, 0.69312102f);
  p = fmaf(p, f, 0.99992448f);
  return __int_as_float(__float_as_int(p) + (__float_as_int(t) << 23));
}

// Soft-cap of attention scores in 32-bit accuracy: cap2 tanh(y) with y = s * scale / cap, from
// tanh(y) = 1 - 2 / (1 + e^(2y)); two_k = 2 log2(e) * scale / cap turns a raw score s into 2y log2(e).
__device__ __forceinline__ float soft_cap(float s, float two_k, float cap2) {
  return cap2 - __fdividef(2.f * cap2, 1.f + exp2f(s * two_k));
}

// The same on the FMA pipe alone for |y| <= SOFT_CAP_POLY_MAX, two scores at a time: tanh(y) / y as a polynomial in y^2,
// fitted at the Chebyshev nodes of [0, SOFT_CAP_POLY_MAX^2] (relative error 2.0e-7 with the fp32 coefficients). k = scale / cap.
constexpr float SOFT_CAP_POLY_MAX = 0.75f;
__device__ __forceinline__ void soft_cap_poly2(float& s0, float& s1, float k, float cap2) {
  float y0, y1, u0, u1, p0, p1;
  mul2(y0, y1, s0, s1, k, k);
  mul2(u0, u1, y0, y1, y0, y1);
  fma2(p0, p1, u0, u1, -0.004723952151834965f, -0.004723952151834965f, 0.01959378644824028f, 0.01959378644824028f);
  fma2(p0, p1, p0, p1, u0, u1, -0.053349819034338f, -0.053349819034338f);
  fma2(p0, p1, p0, p1, u0, u1, 0.13325515389442444f, 0.13325515389442444f);
  fma2(p0, p1, p0, p1, u0, u1, -0.3333296775817871f, -0.3333296775817871f);
  fma2(p0, p1, p0, p1, u0, u1, 1.f, 1.f);
  mul2(y0, y1, y0, y1, cap2, cap2);
  mul2(s0, s1, y0, y1, p0, p1);
}

// The same for |y| <= SOFT_CAP_NEAR_MAX as s * (c0 + c1 s^2 + c2 s^4 + c3 s^6), with scale and cap folded into c (relative
// error 1.6e-7 of the polynomial, fitted likewise).
constexpr float SOFT_CAP_NEAR_MAX = 0.4f;
struct SoftCapNear {
  float c0, c1, c2, c3;
  __device__ __forceinline__ SoftCapNear(float k, float cap2) {
    const float k2 = k * k;
    c0 = cap2 * k;
    c1 = c0 * k2 * -0.3333137333393097f;
    c2 = c0 * k2 * k2 * 0.13271155953407288f;
    c3 = c0 * k2 * k2 * k2 * -0.047561075538396835f;
    c0 *= 0.9999998807907104f;
  }
  __device__ __forceinline__ float at(float s) const {
    const float u = s * s;
    return s * fmaf(fmaf(fmaf(c3, u, c2), u, c1), u, c0);
  }
  // (x0, x1) = at(s0, s1) + (add, add)
  __device__ __forceinline__ void add2(float& x0, float& x1, float s0, float s1, float add) const {
    float u0, u1, p0, p1;
    mul2(u0, u1, s0, s1, s0, s1);
    fma2(p0, p1, u0, u1, c3, c3, c2, c2);
    fma2(p0, p1, p0, p1, u0, u1, c1, c1);
    fma2(p0, p1, p0, p1, u0, u1, c0, c0);
    fma2(x0, x1, s0, s1, p0, p1, add, add);
  }
};

// Epilogue helper: a warp holds a 32-row block one row per lane, each row 128 bytes as eight 16-byte chunks
// (64 bf16 or 32 fp32 values). Writing it straight out would make every store instruction touch 32 different rows
// with 16 bytes each; instead the block goes through a swizzled 4 KB shared-memory stage and leaves as four whole
// 128-byte row segments per instruction. `gbase` points at (first row, first column) of the block in global
// memory, `ld_bytes` is the row pitch, rows >= valid_rows and 16-byte chunks >= valid_chunks are skipped.
// ACC_F32 adds the staged fp32 values to what is in memory (gradient accumulation, fp32 residual streams).
template <bool ACC_F32>
__device__ __forceinline__ void store_rows_coalesced(uint8_t* stage, const uint4 (&pk)[8], uint8_t* gbase,
                                                     long long ld_bytes, int valid_rows, int valid_chunks, int lane) {
#pragma unroll
  for (int j = 0; j < 8; ++j) *reinterpret_cast<uint4*>(stage + lane * 128 + ((j ^ (lane & 7)) << 4)) = pk[j];
  __syncwarp();
  const int ch = lane & 7;
  const bool col_ok = ch < valid_chunks;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int r = i * 4 + (lane >> 3);
    uint4 v = *reinterpret_cast<const uint4*>(stage + r * 128 + ((ch ^ (r & 7)) << 4));
    if (col_ok && r < valid_rows) {
      uint4* g = reinterpret_cast<uint4*>(gbase + r * ld_bytes + ch * 16);
      if (ACC_F32) {   // added in L2: nothing to wait for (every element has one writer, so the sum is reproducible)
        asm volatile("red.global.add.v4.f32 [%0], {%1, %2, %3, %4};" ::"l"(g), "f"(__uint_as_float(v.x)),
                     "f"(__uint_as_float(v.y)), "f"(__uint_as_float(v.z)), "f"(__uint_as_float(v.w))
                     : "memory");
      } else {
        *g = v;
      }
    }
  }
  __syncwarp();
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// Block-wide sum; `red` is a shared array of >= 32 floats. All threads get the result.
__device__ __forceinline__ float block_sum(float v, float* red) {
  int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float t = (lane < nw) ? red[lane] : 0.f;
  t = warp_sum(t);
  return t;
}
__device__ __forceinline__ float block_max(float v, float* red) {
  int lane = threadIdx.x & 31, w = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) red[w] = v;
  __syncthreads();
  float t = (lane < nw) ? red[lane] : -INFINITY;
  t = warp_max(t);
  return t;
}

#endif  // __CUDACC__

}  // namespace edl
