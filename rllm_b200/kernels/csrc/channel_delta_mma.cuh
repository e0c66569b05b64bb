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
//   pass 2 (a chunk after the other)    a block owns 16 value columns of a head; its four warps keep S^T (16 columns
//           x a quarter of the rows each) in registers, as accumulators.  Per chunk: the warps' parts of W S_0 and
//           (q e^G) S_0 meet in shared memory, every warp takes U from them, and the outer products are added to
//           its part of S.  Accumulators become operands without leaving the registers (S^T and U^T are always
//           the left factor); the records come through a ring of three buffers (cp.async).
//
// What is float32 by this design's rules never passes through one bfloat16 number: S, U and every array of a record
// go into a product as the sum of two (value and remainder), the product of the remainders left out: 16 bits of
// mantissa.  Values v are the convolution's activations and exact in bfloat16.
#pragma once
#include "lightning_mma.cuh"

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

__device__ __forceinline__ void cdm_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const bf16 a = __float2bfloat16_rn(x), b = __float2bfloat16_rn(y);
  hi = ltc_pack(a, b);
  lo = ltc_pack(__float2bfloat16_rn(x - __bfloat162float(a)), __float2bfloat16_rn(y - __bfloat162float(b)));
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
  __shared__ float As[CDM_CHUNK][CDM_CHUNK + 1], Bs[CDM_CHUNK][CDM_CHUNK + 1], Xs[CDM_CHUNK][CDM_CHUNK + 1];
  __shared__ float rk[CDM_CHUNK], rq[CDM_CHUNK], bet[CDM_CHUNK];
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, s = blockIdx.y / seg, ci = blockIdx.y % seg;
  const int t0 = q_start[s] + (chunk0 + ci) * CDM_CHUNK;
  const int n = min(CDM_CHUNK, q_start[s + 1] - t0);
  if (n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kvh = h / (heads / kv);
  const float rate = expf(a_log[h]) * 1.4426950408889634f;       // the decays' logarithms to base 2
  for (int e = tid; e < CDM_CHUNK * D; e += CDM_PREP_THREADS) {
    const int i = e / D, x = e - i * D;
    const bool on = i < n && x < d;
    const bf16* row = c + (size_t)(t0 + i) * c_stride;
    qf[i][x] = on ? __bfloat162float(row[(size_t)kvh * d + x]) : 0.f;
    kf[i][x] = on ? __bfloat162float(row[(size_t)(kv + kvh) * d + x]) : 0.f;
    float l = 0.f;
    if (on) {
      const float z = step[((size_t)(t0 + i) * heads + h) * d + x] + dt_bias[h * d + x];
      l = -rate * (z > 20.f ? z : log1pf(expf(z)));
    }
    G[i][x] = l;
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
    float a[2][2] = {}, bb[2][2] = {};
#pragma unroll 1
    for (int u = 0; u < D / 32; ++u) {
      const int x = 4 * (sl + 8 * u);
      float ki[2][4], qi[2][4], gi[2][4], kj[2][4], gj[2][4];
#pragma unroll
      for (int p = 0; p < 2; ++p) {
        *(float4*)ki[p] = *(const float4*)&kf[i0 + p][x];
        *(float4*)qi[p] = *(const float4*)&qf[i0 + p][x];
        *(float4*)gi[p] = *(const float4*)&G[i0 + p][x];
        *(float4*)kj[p] = *(const float4*)&kf[j0 + p][x];
        *(float4*)gj[p] = *(const float4*)&G[j0 + p][x];
      }
#pragma unroll
      for (int p = 0; p < 2; ++p)
#pragma unroll
        for (int r = 0; r < 2; ++r)
#pragma unroll
          for (int y = 0; y < 4; ++y) {
            const float w = kj[r][y] * exp2f(fminf(gi[p][y] - gj[r][y], 0.f));
            a[p][r] = fmaf(ki[p][y], w, a[p][r]);
            bb[p][r] = fmaf(qi[p][y], w, bb[p][r]);
          }
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
        Xs[i][lane] = x[i];
      }
    }
  } else {
    const int t = tid - 32;
    constexpr int N = CDM_PREP_THREADS - 32;
    for (int e = t; e < CDM_CHUNK * D / 2; e += N) {
      const int i = e / (D / 2), x = 2 * (e - i * (D / 2));
      const float g0 = G[i][x], g1 = G[i][x + 1], z0 = G[CDM_CHUNK - 1][x], z1 = G[CDM_CHUNK - 1][x + 1];
      const float e0 = exp2f(g0), e1 = exp2f(g1);
      const float k0 = kf[i][x] * rk[i], k1 = kf[i][x + 1] * rk[i];
      uint32_t hi, lo;
      cdm_split2(qf[i][x] * rq[i] * e0, qf[i][x + 1] * rq[i] * e1, hi, lo);
      *(uint32_t*)&R.qh[i][x] = hi;
      *(uint32_t*)&R.ql[i][x] = lo;
      cdm_split2(k0 * exp2f(z0 - g0), k1 * exp2f(z1 - g1), hi, lo);
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
    for (int x = t; x < D; x += N) R.eg[x] = exp2f(G[CDM_CHUNK - 1][x]);
  }
  __syncthreads();
  for (int e = tid; e < 4 * (D / 2); e += CDM_PREP_THREADS) {      // four tokens of two channels
    const int qd = e / (D / 2), x = 2 * (e - qd * (D / 2));
    float w0[4] = {}, w1[4] = {};
    for (int j = 0; j < 4 * qd + 4; ++j) {
      const float2 k2 = *(const float2*)&kf[j][x];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const float f = Xs[4 * qd + p][j];         // (zero above the diagonal)
        w0[p] = fmaf(f, k2.x, w0[p]);
        w1[p] = fmaf(f, k2.y, w1[p]);
      }
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
  for (int col = tid; col < dvp; col += CDM_PREP_THREADS) {        // a value column's sixteen tokens
    float v[CDM_CHUNK];
#pragma unroll
    for (int j = 0; j < CDM_CHUNK; ++j)
      v[j] = (j < n && col < dv) ? __bfloat162float(c[(size_t)(t0 + j) * c_stride + 2 * (size_t)kv * d + (size_t)h * dv + col]) : 0.f;
#pragma unroll
    for (int i4 = 0; i4 < CDM_CHUNK / 4; ++i4) {
      float o[4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        o[p] = 0.f;
#pragma unroll
        for (int j = 0; j <= 4 * i4 + p; ++j) o[p] = fmaf(Xs[4 * i4 + p][j], v[j], o[p]);
      }
      *(float4*)(ub + (size_t)col * CDM_CHUNK + 4 * i4) = make_float4(o[0], o[1], o[2], o[3]);
    }
  }
}

// Pass 2.  Grid (16-column groups, heads, sequences), four warps; warp w owns rows w * D / 4 .. of S.
template <int D>
__global__ void __launch_bounds__(128)
channel_delta_chunks_kernel(const CdmRecord<D>* rec, const float* u0, float* state, const int* q_start, const int* slots,
                            int num_slots, int chunk0, int seg, float* out, int heads, int d, int dv, int dvp, int* err) {
  constexpr int KS = D / 64;                       // 16-row steps a warp
  constexpr int NT = 2 * KS;                       // 8-row tiles a warp
  extern __shared__ __align__(16) unsigned char cdm_raw[];
  CdmRecord<D>* ring = reinterpret_cast<CdmRecord<D>*>(cdm_raw);
  float4* part = reinterpret_cast<float4*>(cdm_raw + CDM_STAGES * sizeof(CdmRecord<D>));   // [warp][4][32]
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
  const int r0 = warp * (D / 4);
  const size_t unit0 = (size_t)s * seg * heads + h;              // record of chunk x: unit0 + x * heads
  auto fetch = [&](int x) {
    if (x < chunks) {
      const unsigned char* src = reinterpret_cast<const unsigned char*>(rec + unit0 + (size_t)x * heads);
      const unsigned dst = (unsigned)__cvta_generic_to_shared(ring + x % CDM_STAGES);
      for (int e = tid; e < (int)(sizeof(CdmRecord<D>) / 16); e += 128)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst + 16 * e), "l"(src + 16 * e) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int x = 0; x < CDM_STAGES - 1; ++x) fetch(x);
  float* sp = state + ((size_t)slot * heads + h) * d * dv;
  float S[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = r0 + nt * 8 + 2 * tq + (x & 1), col = col0 + g + 8 * (x >> 1);
      S[nt][x] = (row < d && col < dv) ? sp[(size_t)row * dv + col] : 0.f;
    }
  float2 un[4];                                    // the next chunk's U_0: columns g, g + 8 by token pairs 2 tq, 8 + 2 tq
  auto fetch_u = [&](int x) {
    const float* ub = u0 + (unit0 + (size_t)x * heads) * dvp * CDM_CHUNK + (size_t)(col0 + g) * CDM_CHUNK + 2 * tq;
    un[0] = *(const float2*)ub;
    un[1] = *(const float2*)(ub + 8 * CDM_CHUNK);
    un[2] = *(const float2*)(ub + 8);
    un[3] = *(const float2*)(ub + 8 * CDM_CHUNK + 8);
  };
  fetch_u(0);
  for (int ch = 0; ch < chunks; ++ch) {
    asm volatile("cp.async.wait_group %0;" ::"n"(CDM_STAGES - 2) : "memory");
    __syncthreads();                               // this chunk's record is in; the one before it is done with
    fetch(ch + CDM_STAGES - 1);
    const CdmRecord<D>& R = ring[ch % CDM_STAGES];
    float P[2][4] = {}, O[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
      uint32_t ah[4], al[4], bh[4], bl[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) cdm_split2(S[2 * ks + (x >> 1)][2 * (x & 1)], S[2 * ks + (x >> 1)][2 * (x & 1) + 1], ah[x], al[x]);
      ltc_b<D + 8>(bh, &R.wh[0][0], 0, r0 + 16 * ks);
      ltc_b<D + 8>(bl, &R.wl[0][0], 0, r0 + 16 * ks);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        tgm_mma(P[nt], ah, bh[2 * nt], bh[2 * nt + 1]);
        tgm_mma(P[nt], al, bh[2 * nt], bh[2 * nt + 1]);
        tgm_mma(P[nt], ah, bl[2 * nt], bl[2 * nt + 1]);
      }
      ltc_b<D + 8>(bh, &R.qh[0][0], 0, r0 + 16 * ks);
      ltc_b<D + 8>(bl, &R.ql[0][0], 0, r0 + 16 * ks);
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        tgm_mma(O[nt], ah, bh[2 * nt], bh[2 * nt + 1]);
        tgm_mma(O[nt], al, bh[2 * nt], bh[2 * nt + 1]);
        tgm_mma(O[nt], ah, bl[2 * nt], bl[2 * nt + 1]);
      }
    }
    part[(warp * 4 + 0) * 32 + lane] = make_float4(P[0][0], P[0][1], P[0][2], P[0][3]);
    part[(warp * 4 + 1) * 32 + lane] = make_float4(P[1][0], P[1][1], P[1][2], P[1][3]);
    part[(warp * 4 + 2) * 32 + lane] = make_float4(O[0][0], O[0][1], O[0][2], O[0][3]);
    part[(warp * 4 + 3) * 32 + lane] = make_float4(O[1][0], O[1][1], O[1][2], O[1][3]);
    __syncthreads();
    // U^T = U_0^T - the four warps' parts, in every warp (fragment layouts are the same: a lane reads its own places)
    float U[2][4] = {{un[0].x, un[0].y, un[1].x, un[1].y}, {un[2].x, un[2].y, un[3].x, un[3].y}};
    if (ch + 1 < chunks) fetch_u(ch + 1);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float4 p = part[(w * 4 + nt) * 32 + lane];
        U[nt][0] -= p.x; U[nt][1] -= p.y; U[nt][2] -= p.z; U[nt][3] -= p.w;
      }
    uint32_t uh[4], ul[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) cdm_split2(U[x >> 1][2 * (x & 1)], U[x >> 1][2 * (x & 1) + 1], uh[x], ul[x]);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const float2 e = *(const float2*)&R.eg[r0 + nt * 8 + 2 * tq];
      S[nt][0] *= e.x; S[nt][1] *= e.y; S[nt][2] *= e.x; S[nt][3] *= e.y;
    }
#pragma unroll
    for (int np = 0; np < KS; ++np) {
      uint32_t bh[4], bl[4];
      ltc_b_t<D + 8>(bh, &R.kh[0][0], r0 + np * 16, 0);
      ltc_b_t<D + 8>(bl, &R.kl[0][0], r0 + np * 16, 0);
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        tgm_mma(S[2 * np + y], uh, bh[2 * y], bh[2 * y + 1]);
        tgm_mma(S[2 * np + y], ul, bh[2 * y], bh[2 * y + 1]);
        tgm_mma(S[2 * np + y], uh, bl[2 * y], bl[2 * y + 1]);
      }
    }
    if (warp < 2) {                                // the outputs of tokens 8 warp .. + 7
      float o[4] = {};
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float4 p = part[(w * 4 + 2 + warp) * 32 + lane];
        o[0] += p.x; o[1] += p.y; o[2] += p.z; o[3] += p.w;
      }
      uint32_t bh[4], bl[4];
      ltc_b<CDM_BLD>(bh, &R.bh[0][0], 0, 0);
      ltc_b<CDM_BLD>(bl, &R.bl[0][0], 0, 0);
      const uint32_t h0 = warp ? bh[2] : bh[0], h1 = warp ? bh[3] : bh[1], l0 = warp ? bl[2] : bl[0], l1 = warp ? bl[3] : bl[1];
      tgm_mma(o, uh, h0, h1);
      tgm_mma(o, ul, h0, h1);
      tgm_mma(o, uh, l0, l1);
      const int t = (chunk0 + ch) * CDM_CHUNK + 8 * warp + 2 * tq;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int tt = t + (x & 1), col = col0 + g + 8 * (x >> 1);
        if (tt < len && col < dv) out[((size_t)(first + tt) * heads + h) * dv + col] = o[x];
      }
    }
  }
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = r0 + nt * 8 + 2 * tq + (x & 1), col = col0 + g + 8 * (x >> 1);
      if (row < d && col < dv) sp[(size_t)row * dv + col] = S[nt][x];
    }
}
