// What the tcgen05 attention kernels share: the softmax warps' arithmetic, the exchange between the two threads of a
// row, and the host's tensor maps.
#pragma once
#include "tcgen05.cuh"
#include <math.h>

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int x, int y, int z, void* bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];"
               ::"r"(tg_smem(dst)), "l"((unsigned long long)map), "r"(x), "r"(y), "r"(z), "r"(tg_smem(bar)) : "memory");
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));   // rcp(+inf) = +0
  return y;
}
__device__ __forceinline__ float at_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// The softmax warps' arithmetic uses the instructions of sm_100 that do two float32 operations
// (fma.rn.f32x2, add.rn.f32x2 on register pairs) or take three inputs (max.f32): a quarter fewer
// instructions a tile (measured: 2 to 3 % less time at 8,192 tokens; the exponentials and the
// hand-overs between warps weigh more).
__device__ __forceinline__ float at_max3(float a, float b, float c) {
  float d;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(d) : "f"(a), "f"(b), "f"(c));
  return d;
}
__device__ __forceinline__ unsigned long long at_pack2(float lo, float hi) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void at_unpack2(unsigned long long v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ unsigned long long at_fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long at_add2(unsigned long long a, unsigned long long b) {
  unsigned long long d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// 2^x for two numbers at once without the special-function unit: x = n + f with n whole and |f| <= 1/2 (the
// 1.5 * 2^23 trick), a polynomial of degree 4 for 2^f (relative error 4e-5, far below bfloat16's step), and n
// added into the exponent bits.  x below -126 gives 2^-126 (as good as 0 beside a sum that is at least 2^-8).
__device__ __forceinline__ void at_exp2_poly2(unsigned long long x2, float& r0, float& r1) {
  float x0, x1;
  at_unpack2(x2, x0, x1);
  x2 = at_pack2(fmaxf(x0, -126.0f), fmaxf(x1, -126.0f));
  const unsigned long long magic = at_pack2(12582912.0f, 12582912.0f), nmagic = at_pack2(-12582912.0f, -12582912.0f);
  const unsigned long long t2 = at_add2(x2, magic);
  const unsigned long long n2 = at_add2(t2, nmagic);
  const unsigned long long f2 = at_fma2(n2, at_pack2(-1.0f, -1.0f), x2);
  unsigned long long p2 = at_fma2(at_pack2(0.0096181291f, 0.0096181291f), f2, at_pack2(0.0555041087f, 0.0555041087f));
  p2 = at_fma2(p2, f2, at_pack2(0.2402265070f, 0.2402265070f));
  p2 = at_fma2(p2, f2, at_pack2(0.6931471806f, 0.6931471806f));
  p2 = at_fma2(p2, f2, at_pack2(1.0f, 1.0f));
  float p0, p1, t0, t1;
  at_unpack2(p2, p0, p1);
  at_unpack2(t2, t0, t1);
  r0 = __uint_as_float(__float_as_uint(p0) + (__float_as_uint(t0) << 23));
  r1 = __uint_as_float(__float_as_uint(p1) + (__float_as_uint(t1) << 23));
}

// Two CTAs fit one SM, so that one CTA's softmax runs beside the other's products.
// The two threads of a row (one in warp w, one in warp w + 4, same TMEM lane) swap one value:
// each stores its own into a column of its own (`t_mine`, among the score columns it has read) and
// reads the other's (`t_theirs`) after the pair's mbarrier (two arrivals, one a warp; exchange n
// completes phase n).  Exchanges take two columns in turn: a column is used again two exchanges
// later at the earliest, when the partner, having passed the barrier between, has read it.  The
// columns may be score columns that the thread has read: the next tile's scores are written over
// them only after both have told the MMA warp that they are through with the tile.  False if the
// wait ran out.
__device__ __forceinline__ bool pair_exchange(unsigned t_mine, unsigned t_theirs, void* bar, int n, float mine, float* theirs, int* err) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x1.b32 [%0], {%1};" ::"r"(t_mine), "r"(__float_as_uint(mine)) : "memory");
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncwarp();
  if ((threadIdx.x & 31) == 0) mbar_arrive(bar);
  if (!__all_sync(0xffffffffu, mbar_wait(bar, n & 1, err))) return false;
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  unsigned other;
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x1.b32 {%0}, [%1];" : "=r"(other) : "r"(t_theirs) : "memory");
  asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
  *theirs = __uint_as_float(other);
  return true;
}

static int at_encode(CUtensorMap* map, int rank, const void* ptr, const cuuint64_t* dims, const cuuint64_t* strides,
                     const cuuint32_t* box) {
  tg_encode_fn enc = tg_get_encode();
  if (!enc) return RLLM_E_UNSUPPORTED;
  cuuint32_t estr[3] = {1, 1, 1};
  CUresult r = enc(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, (cuuint32_t)rank, const_cast<void*>(ptr), dims, strides, box,
                   estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? 0 : RLLM_E_BADARG;
}
