// The delta rule of channel_delta.cu over long portions of bfloat16 activations, sixteen tokens at a time on the
// tensor cores (mma.sync m16n8k16, float32 accumulators).  With G_i the sum of the logarithms of the decays of a
// chunk's tokens up to i (per key channel) and S_0 the state ahead of the chunk, the recurrence unrolls to
//
//   u_i = beta_i (v_i - (k_i e^{G_i})^T S_0 - sum_{j < i} A_ij u_j),     A_ij = sum_c k_ic k_jc e^{G_ic - G_jc}
//   o_i = (q_i e^{G_i})^T S_0 + sum_{j <= i} B_ij u_j,                   B_ij = sum_c q_ic k_jc e^{G_ic - G_jc}
//   S_C = diag(e^{G_C}) S_0 + sum_j (k_j e^{G_C - G_j}) u_j^T
//
// and with X = (I + diag(beta) A)^{-1} diag(beta) (forward substitution, 16 x 16), W = X (k e^G), U_0 = X V:
//   U = U_0 - W S_0.   Every exponent is a sum of logarithms of decays between two tokens: none is positive.
//
//   pass 1 (all chunks side by side)    makes a chunk's record: W, q e^G, k e^{G_C - G}, B, e^{G_C}; and U_0
//   pass 2 (a chunk after the other)    a block owns 16 value columns of a head; four of its warps keep S^T (16
//           columns x a quarter of the rows each) in registers, as accumulators.  Per chunk: their parts of W S_0
//           meet in shared memory, each takes U from them and adds the outer products to its part of S.
//           Accumulators become operands without leaving the registers (S^T and U^T are always the left factor).
//           Two more warps make the outputs a step behind; one brings the records through a ring of three buffers
//           (bulk copies that complete on an mbarrier).
//
// What is float32 by this design's rules never passes through one bfloat16 number: S, U and every array of a record
// go into a product as the sum of two (value and remainder), the product of the remainders left out: 16 bits of
// mantissa.  Values v are the convolution's activations and exact in bfloat16.
#pragma once
#include "lightning_mma.cuh"
#include "tcgen05.cuh"

#define CDM_CHUNK 16
#define CDM_STAGES 3
#define CDM_BLD 24              // row length of the two 16 x 16 arrays in a record

// A chunk's record, as it lies in global and in shared memory (rows of D + 8: ldmatrix without bank conflicts)
template <int D> struct alignas(16) CdmRecord {
  bf16 wh[CDM_CHUNK][D + 8], wl[CDM_CHUNK][D + 8];
  bf16 qh[CDM_CHUNK][D + 8], ql[CDM_CHUNK][D + 8];
  bf16 kh[CDM_CHUNK][D + 8], kl[CDM_CHUNK][D + 8];
  bf16 bh[CDM_CHUNK][CDM_BLD], bl[CDM_CHUNK][CDM_BLD];
  float eg[D];
};

// (x, y) as packed values and packed remainders
__device__ __forceinline__ void cdm_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  hi = *(const uint32_t*)&h;
  lo = *(const uint32_t*)&l;
}
// 2^x for x <= 0 (one special-function operation; results below the normal range become zero)
__device__ __forceinline__ float cdm_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// log2(e) softplus(z) for the logarithms of decays: e = 2^(z log2 e), then log2(1 + e), by its series where 1 + e
// would round e away
__device__ __forceinline__ float cdm_softplus_log2(float z) {
  const float x = z * 1.4426950408889634f;
  if (z > 20.f) return x;
  float e, l;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x));
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.0f + e));
  const float series = e * fmaf(e, fmaf(e, fmaf(e, fmaf(e, 0.2f, -0.25f), 0.33333333f), -0.5f), 1.0f);
  return e < 0.0625f ? series * 1.4426950408889634f : l;
}
// two float32 sums, products and multiply-adds an instruction
__device__ __forceinline__ unsigned long long cdm_pack(float x, float y) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ float2 cdm_unpack(unsigned long long v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ unsigned long long cdm_fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ unsigned long long cdm_mul2(unsigned long long a, unsigned long long b) {
  unsigned long long r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// Pass 1.  Grid (heads, sequences * seg); 36 tiles of 2 x 2 token pairs (the lower triangle) by 8 slices of the
// channels.
#define CDM_PREP_THREADS 288
template <int D>
__global__ void __launch_bounds__(CDM_PREP_THREADS, 3)
channel_delta_records_kernel(const bf16* c, int c_stride, const float* step, const float* b, const float* dt_bias,
                             const float* a_log, const int* q_start, int chunk0, int seg, CdmRecord<D>* rec, float* u0,
                             int heads, int kv, int d, int dv, int dvp, float unit_eps, float qscale) {
  constexpr int LD = D + 4;
  __shared__ __align__(16) float kf[CDM_CHUNK][LD], qf[CDM_CHUNK][LD], G[CDM_CHUNK][LD];
  __shared__ float As[CDM_CHUNK][CDM_CHUNK + 1], Bs[CDM_CHUNK][CDM_CHUNK + 1];
  __shared__ __align__(16) float Xt[CDM_CHUNK][CDM_CHUNK + 4];     // X transposed: [column][row]
  __shared__ float rk[CDM_CHUNK], rq[CDM_CHUNK], bet[CDM_CHUNK];
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, s = blockIdx.y / seg, ci = blockIdx.y % seg;
  const int t0 = q_start[s] + (chunk0 + ci) * CDM_CHUNK;
  const int n = min(CDM_CHUNK, q_start[s + 1] - t0);
  if (n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kvh = h / (heads / kv);
  const float rate = expf(a_log[h]);                               // (the decays' logarithms are to base 2)
  const bool even = ((d | c_stride) & 1) == 0;                     // two channels a load
  for (int e = tid; e < CDM_CHUNK * D / 2; e += CDM_PREP_THREADS) {
    const int i = e / (D / 2), x = 2 * (e - i * (D / 2));
    const bf16* row = c + (size_t)(t0 + i) * c_stride;
    float2 qv = make_float2(0.f, 0.f), kv2 = qv, z = qv, l = qv;
    if (i < n && x < d) {
      const float* st = step + ((size_t)(t0 + i) * heads + h) * d + x;
      if (even) {
        qv = __bfloat1622float2(*(const __nv_bfloat162*)(row + (size_t)kvh * d + x));
        kv2 = __bfloat1622float2(*(const __nv_bfloat162*)(row + (size_t)(kv + kvh) * d + x));
        z = *(const float2*)st;
      } else {
        qv.x = __bfloat162float(row[(size_t)kvh * d + x]);
        kv2.x = __bfloat162float(row[(size_t)(kv + kvh) * d + x]);
        z.x = st[0];
        if (x + 1 < d) {
          qv.y = __bfloat162float(row[(size_t)kvh * d + x + 1]);
          kv2.y = __bfloat162float(row[(size_t)(kv + kvh) * d + x + 1]);
          z.y = st[1];
        }
      }
      z.x += dt_bias[h * d + x];
      l.x = -rate * cdm_softplus_log2(z.x);
      if (x + 1 < d) {
        z.y += dt_bias[h * d + x + 1];
        l.y = -rate * cdm_softplus_log2(z.y);
      }
    }
    *(float2*)&qf[i][x] = qv;
    *(float2*)&kf[i][x] = kv2;
    *(float2*)&G[i][x] = l;
  }
  if (tid < CDM_CHUNK) bet[tid] = tid < n ? 1.0f / (1.0f + expf(-b[(size_t)(t0 + tid) * heads + h])) : 0.f;
  __syncthreads();
  for (int it = warp; it < 2 * CDM_CHUNK; it += CDM_PREP_THREADS / 32) {
    const int i = it >> 1;
    const float* row = (it & 1) ? kf[i] : qf[i];
    float ss = 0.f;
    for (int x = lane; x < D; x += 32) ss = fmaf(row[x], row[x], ss);
    ss = warp_sum(ss);
    if (lane == 0) { if (it & 1) rk[i] = 1.0f / sqrtf(ss + unit_eps); else rq[i] = qscale / sqrtf(ss + unit_eps); }
  }
  for (int x = tid; x < D; x += CDM_PREP_THREADS) {
    float run = 0.f;
#pragma unroll
    for (int i = 0; i < CDM_CHUNK; ++i) { run += G[i][x]; G[i][x] = run; }
  }
  __syncthreads();
  {
    // tile number -> (row tile, column tile) of the lower triangle; lanes of one tile are neighbours
    const int tile = tid >> 3, sl = tid & 7;
    int ti = 0;
    while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
    const int tj = tile - ti * (ti + 1) / 2, i0 = 2 * ti, j0 = 2 * tj;
    unsigned long long a2[2][2] = {}, b2[2][2] = {};           // sums over even and odd channels
#pragma unroll 1
    for (int u = 0; u < D / 32; ++u) {
      const int x = 4 * (sl + 8 * u);
      ulonglong2 ki[2], qi[2], kj[2];
      float gi[2][4], gj[2][4];
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        ki[p] = *(const ulonglong2*)&kf[i0 + p][x];
        qi[p] = *(const ulonglong2*)&qf[i0 + p][x];
        kj[p] = *(const ulonglong2*)&kf[j0 + p][x];
        *(float4*)gi[p] = *(const float4*)&G[i0 + p][x];
        *(float4*)gj[p] = *(const float4*)&G[j0 + p][x];
      }
#pragma unroll
      for (int p = 0; p < 2; ++p)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          // (a pair above the diagonal has rising exponents: its sums are thrown away)
          const unsigned long long e0 = cdm_pack(cdm_exp2(gi[p][0] - gj[r][0]), cdm_exp2(gi[p][1] - gj[r][1]));
          const unsigned long long e1 = cdm_pack(cdm_exp2(gi[p][2] - gj[r][2]), cdm_exp2(gi[p][3] - gj[r][3]));
          const unsigned long long w0 = cdm_mul2(kj[r].x, e0), w1 = cdm_mul2(kj[r].y, e1);
          a2[p][r] = cdm_fma2(ki[p].y, w1, cdm_fma2(ki[p].x, w0, a2[p][r]));
          b2[p][r] = cdm_fma2(qi[p].y, w1, cdm_fma2(qi[p].x, w0, b2[p][r]));
        }
    }
    float a[2][2], bb[2][2];
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float2 ua = cdm_unpack(a2[p][r]), ub = cdm_unpack(b2[p][r]);
        a[p][r] = ua.x + ua.y;
        bb[p][r] = ub.x + ub.y;
      }
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) {
          a[p][r] += __shfl_xor_sync(0xffffffffu, a[p][r], o);
          bb[p][r] += __shfl_xor_sync(0xffffffffu, bb[p][r], o);
        }
        const int i = i0 + p, j = j0 + r;
        if (sl == 0) {
          As[i][j] = j < i ? a[p][r] * rk[i] * rk[j] : 0.f;
          Bs[i][j] = j <= i ? bb[p][r] * rq[i] * rk[j] : 0.f;
        }
      }
  }
  __syncthreads();
  CdmRecord<D>& R = rec[(size_t)blockIdx.y * heads + h];
  if (warp == 0) {
    if (lane < CDM_CHUNK) {                        // column `lane` of X
      float x[CDM_CHUNK];
#pragma unroll
      for (int i = 0; i < CDM_CHUNK; ++i) {
        float r = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int l = 0; l < i; ++l) r = fmaf(-As[i][l], x[l], r);
        x[i] = bet[i] * r;
        Xt[lane][i] = x[i];
      }
    }
  } else {
    const int t = tid - 32;
    constexpr int N = CDM_PREP_THREADS - 32;
    for (int e = t; e < CDM_CHUNK * D / 2; e += N) {
      const int i = e / (D / 2), x = 2 * (e - i * (D / 2));
      const float g0 = G[i][x], g1 = G[i][x + 1], z0 = G[CDM_CHUNK - 1][x], z1 = G[CDM_CHUNK - 1][x + 1];
      const float e0 = cdm_exp2(g0), e1 = cdm_exp2(g1);
      const float k0 = kf[i][x] * rk[i], k1 = kf[i][x + 1] * rk[i];
      uint32_t hi, lo;
      cdm_split2(qf[i][x] * rq[i] * e0, qf[i][x + 1] * rq[i] * e1, hi, lo);
      *(uint32_t*)&R.qh[i][x] = hi;
      *(uint32_t*)&R.ql[i][x] = lo;
      cdm_split2(k0 * cdm_exp2(z0 - g0), k1 * cdm_exp2(z1 - g1), hi, lo);
      *(uint32_t*)&R.kh[i][x] = hi;
      *(uint32_t*)&R.kl[i][x] = lo;
      kf[i][x] = k0 * e0;                          // what W is made of
      kf[i][x + 1] = k1 * e1;
    }
    for (int e = t; e < CDM_CHUNK * CDM_CHUNK / 2; e += N) {
      const int i = e >> 3, j = 2 * (e & 7);
      uint32_t hi, lo;                             // (above the diagonal's tiles Bs was not written: zeros)
      cdm_split2(j <= i ? Bs[i][j] : 0.f, j + 1 <= i ? Bs[i][j + 1] : 0.f, hi, lo);
      *(uint32_t*)&R.bh[i][j] = hi;
      *(uint32_t*)&R.bl[i][j] = lo;
    }
    for (int x = t; x < D; x += N) R.eg[x] = cdm_exp2(G[CDM_CHUNK - 1][x]);
  }
  __syncthreads();
  for (int e = tid; e < 4 * (D / 2); e += CDM_PREP_THREADS) {      // four tokens of two channels
    const int qd = e / (D / 2), x = 2 * (e - qd * (D / 2));
    float w0[4] = {}, w1[4] = {};
    for (int j = 0; j < 4 * qd + 4; ++j) {
      const float2 k2 = *(const float2*)&kf[j][x];
      const float4 f4 = *(const float4*)&Xt[j][4 * qd];             // (zero above X's diagonal)
      w0[0] = fmaf(f4.x, k2.x, w0[0]); w1[0] = fmaf(f4.x, k2.y, w1[0]);
      w0[1] = fmaf(f4.y, k2.x, w0[1]); w1[1] = fmaf(f4.y, k2.y, w1[1]);
      w0[2] = fmaf(f4.z, k2.x, w0[2]); w1[2] = fmaf(f4.z, k2.y, w1[2]);
      w0[3] = fmaf(f4.w, k2.x, w0[3]); w1[3] = fmaf(f4.w, k2.y, w1[3]);
    }
#pragma unroll
    for (int p = 0; p < 4; ++p) {
      uint32_t hi, lo;
      cdm_split2(w0[p], w1[p], hi, lo);
      *(uint32_t*)&R.wh[4 * qd + p][x] = hi;
      *(uint32_t*)&R.wl[4 * qd + p][x] = lo;
    }
  }
  float* ub = u0 + ((size_t)blockIdx.y * heads + h) * dvp * CDM_CHUNK;
  for (int e = tid; e < 4 * dvp; e += CDM_PREP_THREADS) {          // four tokens of a value column
    const int i4 = e / dvp, col = e - i4 * dvp;
    const bf16* vr = c + (size_t)t0 * c_stride + 2 * (size_t)kv * d + (size_t)h * dv + col;
    float o[4] = {};
#pragma unroll 4
    for (int j = 0; j < 4 * i4 + 4; ++j) {
      const float v = (j < n && col < dv) ? __bfloat162float(vr[(size_t)j * c_stride]) : 0.f;
      const float4 f4 = *(const float4*)&Xt[j][4 * i4];
      o[0] = fmaf(f4.x, v, o[0]); o[1] = fmaf(f4.y, v, o[1]); o[2] = fmaf(f4.z, v, o[2]); o[3] = fmaf(f4.w, v, o[3]);
    }
    *(float4*)(ub + (size_t)col * CDM_CHUNK + 4 * i4) = make_float4(o[0], o[1], o[2], o[3]);
  }
}

// Pass 2.  Grid (16-column groups, heads, sequences), seven warps.  Warps 0 .. 3 carry the recurrence: warp w owns
// rows w * D / 4 .. of S^T.  Warps 4 and 5 make the outputs of a chunk's tokens 0 .. 7 and 8 .. 15 a step behind, from
// the copies of S_0 and U that the first four leave in shared memory (two of each) and the record's fragments that
// they took into registers.  Warp 6 fetches the records.  At barrier A a chunk's record is in, and so are S_0 and U of
// the chunk before; at barrier B, the first four warps' own, the parts of W S_0 are.
#define CDM_THREADS 224
template <int D> struct CdmSmem {
  CdmRecord<D> ring[CDM_STAGES];                   // (16-byte aligned: bulk copies)
  float4 part[4][2][32];                           // the four warps' parts of W S_0, as fragments
  uint4 s0[2][D / 16][2][32];                      // S_0 as left-factor fragments: value, remainder
  uint4 u[2][2][32];                               // U alike
  unsigned long long full[CDM_STAGES];             // mbarriers: a buffer's record has arrived
};
// all of the block's warps, each from its own place in the code
__device__ __forceinline__ void cdm_barrier_b() { asm volatile("bar.sync 2, 128;" ::: "memory"); }
__device__ __forceinline__ void cdm_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(CDM_THREADS) : "memory"); }

template <int D>
__global__ void __launch_bounds__(CDM_THREADS)
channel_delta_chunks_kernel(const CdmRecord<D>* rec, const float* u0, float* state, const int* q_start, const int* slots,
                            int num_slots, int chunk0, int seg, float* out, int heads, int d, int dv, int dvp, int* err) {
  constexpr int KS = D / 64;                       // 16-row steps a warp
  constexpr int NT = 2 * KS;                       // 8-row tiles a warp
  extern __shared__ __align__(16) unsigned char cdm_raw[];
  CdmSmem<D>& sm = *reinterpret_cast<CdmSmem<D>*>(cdm_raw);
  pdl_wait();
  pdl_launch();
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * 16;
  const int first = q_start[s], len = q_start[s + 1] - first;
  const int chunks = min(seg, (len + CDM_CHUNK - 1) / CDM_CHUNK - chunk0);
  if (chunks <= 0) return;
  const int slot = slots[s];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, 8);
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, tq = lane & 3;
  const size_t unit0 = (size_t)s * seg * heads + h;              // record of chunk x: unit0 + x * heads
  if (tid == 0) {
#pragma unroll
    for (int x = 0; x < CDM_STAGES; ++x) mbar_init(&sm.full[x], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  cdm_barrier();
  if (warp == 6) {                                 // ---- the records: one bulk copy each
    auto fetch = [&](int x, int stage) {
      if (x >= chunks || lane != 0) return;
      mbar_expect_tx(&sm.full[stage], (unsigned)sizeof(CdmRecord<D>));
      asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                   ::"r"(tg_smem(sm.ring + stage)), "l"(rec + unit0 + (size_t)x * heads), "r"((unsigned)sizeof(CdmRecord<D>)),
                     "r"(tg_smem(&sm.full[stage])) : "memory");
    };
#pragma unroll
    for (int x = 0; x < CDM_STAGES - 1; ++x) fetch(x, x);
    int stage = 0, into = CDM_STAGES - 1, parity = 0;
    for (int ch = 0; ch < chunks; ++ch) {
      // (if a wait runs out its error word is set and the walk goes on: nobody is left waiting at a barrier)
      mbar_wait(&sm.full[stage], parity, err);
      if (++stage == CDM_STAGES) { stage = 0; parity ^= 1; }
      __syncwarp();
      cdm_barrier();                               // A
      fetch(ch + CDM_STAGES - 1, into);            // (its buffer's chunk, the one before this, is done with)
      if (++into == CDM_STAGES) into = 0;
      __syncwarp();
    }
    cdm_barrier();                                 // A after the last
    return;
  }
  if (warp >= 4) {                                 // ---- the outputs
    const int half = warp - 4;                     // tokens 8 half .. of a chunk
    uint32_t qh[D / 32][4] = {}, ql[D / 32][4] = {}, bh[4] = {}, bl[4] = {};
    float* orow = out + ((size_t)first * heads + h) * dv + col0 + g;
    const size_t ostep = (size_t)heads * dv;
    auto outputs = [&](int ch) {
      float o[3][4] = {};
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        const uint4 a = sm.s0[ch & 1][ks][0][lane], r = sm.s0[ch & 1][ks][1][lane];
        const uint32_t ah[4] = {a.x, a.y, a.z, a.w}, al[4] = {r.x, r.y, r.z, r.w};
        const int k2 = ks >> 1, y = 2 * (ks & 1);
        tgm_mma(o[0], ah, qh[k2][y], qh[k2][y + 1]);
        tgm_mma(o[1], al, qh[k2][y], qh[k2][y + 1]);
        tgm_mma(o[2], ah, ql[k2][y], ql[k2][y + 1]);
      }
      const uint4 a = sm.u[ch & 1][0][lane], r = sm.u[ch & 1][1][lane];
      const uint32_t uh[4] = {a.x, a.y, a.z, a.w}, ul[4] = {r.x, r.y, r.z, r.w};
      const uint32_t h0 = half ? bh[2] : bh[0], h1 = half ? bh[3] : bh[1], l0 = half ? bl[2] : bl[0], l1 = half ? bl[3] : bl[1];
      tgm_mma(o[0], uh, h0, h1);
      tgm_mma(o[1], ul, h0, h1);
      tgm_mma(o[2], uh, l0, l1);
      const int t = (chunk0 + ch) * CDM_CHUNK + 8 * half + 2 * tq;
      float* op = orow + (size_t)t * ostep;
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (t + (x & 1) < len && col0 + g + 8 * (x >> 1) < dv)
          op[(x & 1) * ostep + 8 * (x >> 1)] = o[0][x] + (o[1][x] + o[2][x]);
    };
    int stage = 0;
    for (int ch = 0; ch < chunks; ++ch) {
      cdm_barrier();                               // A
      if (ch > 0) outputs(ch - 1);
      const CdmRecord<D>& R = sm.ring[stage];
      stage = stage + 1 == CDM_STAGES ? 0 : stage + 1;
#pragma unroll
      for (int k2 = 0; k2 < D / 32; ++k2) {        // two 16-row steps of this warp's eight tokens a load
        const int at = (lane & 7) * (D + 8) + 32 * k2 + (lane >> 3) * 8;
        tgm_ldmatrix4(qh[k2], &R.qh[8 * half][0] + at);
        tgm_ldmatrix4(ql[k2], &R.ql[8 * half][0] + at);
      }
      ltc_b<CDM_BLD>(bh, &R.bh[0][0], 0, 0);
      ltc_b<CDM_BLD>(bl, &R.bl[0][0], 0, 0);
    }
    cdm_barrier();                                 // A after the last
    outputs(chunks - 1);
    return;
  }
  // ---- the recurrence
  const int r0 = warp * (D / 4);
  float* sp = state + ((size_t)slot * heads + h) * d * dv;
  float S[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = r0 + nt * 8 + 2 * tq + (x & 1), col = col0 + g + 8 * (x >> 1);
      S[nt][x] = (row < d && col < dv) ? sp[(size_t)row * dv + col] : 0.f;
    }
  // the next chunk's U_0: columns g, g + 8 by token pairs 2 tq, 8 + 2 tq
  float2 un[4];
  const float* ub = u0 + unit0 * dvp * CDM_CHUNK + (size_t)(col0 + g) * CDM_CHUNK + 2 * tq;
  const size_t ustep = (size_t)heads * dvp * CDM_CHUNK;
  auto fetch_u = [&]() {
    un[0] = *(const float2*)ub;
    un[1] = *(const float2*)(ub + 8 * CDM_CHUNK);
    un[2] = *(const float2*)(ub + 8);
    un[3] = *(const float2*)(ub + 8 * CDM_CHUNK + 8);
    ub += ustep;
  };
  fetch_u();
  int stage = 0;
  for (int ch = 0; ch < chunks; ++ch) {
    uint32_t ah[KS][4], al[KS][4];
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int x = 0; x < 4; ++x)
        cdm_split2(S[2 * ks + (x >> 1)][2 * (x & 1)], S[2 * ks + (x >> 1)][2 * (x & 1) + 1], ah[ks][x], al[ks][x]);
    cdm_barrier();                               // A
    const CdmRecord<D>& R = sm.ring[stage];
    stage = stage + 1 == CDM_STAGES ? 0 : stage + 1;
    float P[2][2][4] = {};                         // W S_0: tokens 0 .. 7 and 8 .. 15, the value's product and the rest
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t wh[4], wl[4];
      ltc_b<D + 8>(wh, &R.wh[0][0], 0, r0 + 16 * ks);
      ltc_b<D + 8>(wl, &R.wl[0][0], 0, r0 + 16 * ks);
      // (the products of one sum have others between them: none waits for the one ahead)
      tgm_mma(P[0][0], ah[ks], wh[0], wh[1]); tgm_mma(P[1][0], ah[ks], wh[2], wh[3]);
      tgm_mma(P[0][1], al[ks], wh[0], wh[1]); tgm_mma(P[1][1], al[ks], wh[2], wh[3]);
      tgm_mma(P[0][0], ah[ks], wl[0], wl[1]); tgm_mma(P[1][0], ah[ks], wl[2], wl[3]);
      sm.s0[ch & 1][warp * KS + ks][0][lane] = make_uint4(ah[ks][0], ah[ks][1], ah[ks][2], ah[ks][3]);
      sm.s0[ch & 1][warp * KS + ks][1][lane] = make_uint4(al[ks][0], al[ks][1], al[ks][2], al[ks][3]);
    }
#pragma unroll
    for (int x = 0; x < 2; ++x)
      sm.part[warp][x][lane] = make_float4(P[x][0][0] + P[x][1][0], P[x][0][1] + P[x][1][1], P[x][0][2] + P[x][1][2],
                                           P[x][0][3] + P[x][1][3]);
    // what does not need U: the outer products' right factors, and S decayed
    uint32_t kh[KS][4], kl[KS][4];
#pragma unroll
    for (int np = 0; np < KS; ++np) {
      ltc_b_t<D + 8>(kh[np], &R.kh[0][0], r0 + np * 16, 0);
      ltc_b_t<D + 8>(kl[np], &R.kl[0][0], r0 + np * 16, 0);
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const float2 e = *(const float2*)&R.eg[r0 + nt * 8 + 2 * tq];
      S[nt][0] *= e.x; S[nt][1] *= e.y; S[nt][2] *= e.x; S[nt][3] *= e.y;
    }
    cdm_barrier_b();                             // B
    // U^T = U_0^T - the four warps' parts, in every warp (fragment layouts are the same: a lane reads its own places)
    float U[2][4] = {{un[0].x, un[0].y, un[1].x, un[1].y}, {un[2].x, un[2].y, un[3].x, un[3].y}};
    if (ch + 1 < chunks) fetch_u();
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      const float4 p0 = sm.part[0][nt][lane], p1 = sm.part[1][nt][lane], p2 = sm.part[2][nt][lane], p3 = sm.part[3][nt][lane];
      U[nt][0] -= (p0.x + p1.x) + (p2.x + p3.x); U[nt][1] -= (p0.y + p1.y) + (p2.y + p3.y);
      U[nt][2] -= (p0.z + p1.z) + (p2.z + p3.z); U[nt][3] -= (p0.w + p1.w) + (p2.w + p3.w);
    }
    uint32_t uh[4], ul[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) cdm_split2(U[x >> 1][2 * (x & 1)], U[x >> 1][2 * (x & 1) + 1], uh[x], ul[x]);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) tgm_mma(S[nt], uh, kh[nt >> 1][2 * (nt & 1)], kh[nt >> 1][2 * (nt & 1) + 1]);
    if (warp == 0) {
      sm.u[ch & 1][0][lane] = make_uint4(uh[0], uh[1], uh[2], uh[3]);
      sm.u[ch & 1][1][lane] = make_uint4(ul[0], ul[1], ul[2], ul[3]);
    }
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) tgm_mma(S[nt], ul, kh[nt >> 1][2 * (nt & 1)], kh[nt >> 1][2 * (nt & 1) + 1]);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) tgm_mma(S[nt], uh, kl[nt >> 1][2 * (nt & 1)], kl[nt >> 1][2 * (nt & 1) + 1]);
  }
  cdm_barrier();                                 // A after the last
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = r0 + nt * 8 + 2 * tq + (x & 1), col = col0 + g + 8 * (x >> 1);
      if (row < d && col < dv) sp[(size_t)row * dv + col] = S[nt][x];
    }
}
