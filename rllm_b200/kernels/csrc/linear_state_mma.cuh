// The recurrence of linear_state.cu over long portions of bfloat16 activations, in chunks of C = 64 tokens that run side
// by side on the tensor cores (mma.sync m16n8k16, float32 accumulators).  With G_t the sum of the base-2 logarithms of
// the decays of a chunk's tokens up to t (per channel; fixed decays: (t + 1) log2 lambda) and S_0 the state ahead of the
// chunk:
//
//   pass 1   Z = (K * 2^(G_last - G))^T V                    a chunk's end state from a zero start
//   chain    S_0 of chunk c + 1 = 2^(G_last) * (S_0 of chunk c) + Z     (rows; in order; and the sequence's new state)
//   pass 2   O = (Q * 2^G) S_0 + A V,   A_tj = sum_c q_tc k_jc 2^(G_tc - G_jc) for j <= t, else 0
//            and y from O: a block has all of a head's columns
//
// No exponent is positive, so decays of any strength stay in range.  A with decays per channel: sixteen tokens are a
// block; between blocks I > J a product of Q * 2^(G - G_J) and K * 2^(G_J - G), G_J the sums at the end of block J; inside
// a block pair by pair on the CUDA cores.  With fixed decays: Q K^T times lambda^(t - j).
//
// What enters the recurrence is float32 by this design's rules and never passes through one bfloat16 number: rotated
// queries and keys, q 2^G, the weighted keys, S_0 and A go into their products as the sum of two (value and remainder),
// the product of two remainders left out: 16 bits of mantissa.  Values v are the projections and exact in bfloat16.
#pragma once
#include "linear_state.cuh"
#include "channel_delta_mma.cuh"      // fragment loads, splits and packed conversions

#define LSM_C 64

// rotation table of a step's tokens: cosine and sine per (token, pair)
__global__ void __launch_bounds__(256)
ls_rotation_table_kernel(const int* positions, const double* inv_freq, int half, float2* table, long long n) {
  pdl_wait();
  pdl_launch();
  const long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (e >= n) return;
  float c, s;
  rope_cos_sin(positions[e / half], inv_freq[e % half], &c, &s);
  table[e] = make_float2(c, s);
}

__device__ __forceinline__ void lsm_split4(const float (&v)[4], bf16* hi, bf16* lo) {
  uint2 h, l;
  cdm_split2(v[0], v[1], h.x, l.x);
  cdm_split2(v[2], v[3], h.y, l.y);
  *(uint2*)hi = h;
  *(uint2*)lo = l;
}

// Fixed decays: the chunk's rotated queries (WITH_Q) and keys, four values at a time: put(token, column, q, k).
template <int D, int NT, bool WITH_Q, typename Put>
__device__ __forceinline__ void lsm_rotated(const bf16* q, const bf16* k, const LsArgs& p, const float2* table, int t0, int n,
                                            bool wide, Put put) {
  const int half = p.rd >> 1, quads = (half + 3) / 4, items = quads + (D - p.rd + 3) / 4;
  for (int e = threadIdx.x; e < LSM_C * items; e += NT) {
    const int j = e / items, u = e - j * items;
    const bool on = j < n;
    const size_t at = (size_t)(t0 + j) * p.stride;
    float qa[4] = {0.f, 0.f, 0.f, 0.f}, ka[4];
    if (u < quads) {
      const int i = u * 4, left = half - i;
      float qb[4] = {0.f, 0.f, 0.f, 0.f}, kb[4];
      if (WITH_Q) { ltc_fetch4<true>(q + at + i, on, wide, left, qa); ltc_fetch4<true>(q + at + half + i, on, wide, left, qb); }
      ltc_fetch4<true>(k + at + i, on, wide, left, ka);
      ltc_fetch4<true>(k + at + half + i, on, wide, left, kb);
      const float2* cs = table + (size_t)(t0 + j) * half + i;
      float qlo[4], qhi[4], klo[4], khi[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float2 r = (on && x < left) ? cs[x] : make_float2(0.f, 0.f);
        qlo[x] = qa[x] * r.x - qb[x] * r.y; qhi[x] = qb[x] * r.x + qa[x] * r.y;
        klo[x] = (ka[x] * r.x - kb[x] * r.y) * p.k_scale; khi[x] = (kb[x] * r.x + ka[x] * r.y) * p.k_scale;
      }
      put(j, i, left, qlo, klo);
      put(j, half + i, left, qhi, khi);
    } else {
      const int i = p.rd + (u - quads) * 4, left = p.d - i;
      if (WITH_Q) ltc_fetch4<true>(q + at + i, on, wide, left, qa);
      ltc_fetch4<true>(k + at + i, on, wide, left, ka);
#pragma unroll
      for (int x = 0; x < 4; ++x) ka[x] *= p.k_scale;
      put(j, i, D - i, qa, ka);
    }
  }
}

// four neighbouring values into a row of two bfloat16 arrays (value, remainder), as far as they exist; columns that are
// no multiple of four go one by one
__device__ __forceinline__ void lsm_put4(bf16* hi, bf16* lo, int col, int left, const float (&v)[4]) {
  if ((col & 3) == 0 && left >= 4) { lsm_split4(v, hi + col, lo + col); return; }
#pragma unroll
  for (int x = 0; x < 4; ++x) {
    if (x < left) {
      const bf16 h = __float2bfloat16_rn(v[x]);
      hi[col + x] = h;
      lo[col + x] = __float2bfloat16_rn(v[x] - __bfloat162float(h));
    }
  }
}

// Decays per channel: four neighbouring channels of a token: key, log2 of the decay
__device__ __forceinline__ void lsm_gate4(const bf16* f, const LsArgs& p, int h, int i, bool on, bool wide, float (&k)[4], float (&lf)[4]) {
  float z[4], lo[4], bi[4];
  const int left = p.d - i;
  ltc_fetch4<true>(f, on, wide, left, z);
  if (wide && left >= 4) {                     // (d is a multiple of four: the vectors' rows are 16-byte aligned)
    const float4 a = *(const float4*)(p.lower + h * p.d + i), b = *(const float4*)(p.f_bias + h * p.d + i);
    lo[0] = a.x; lo[1] = a.y; lo[2] = a.z; lo[3] = a.w;
    bi[0] = b.x; bi[1] = b.y; bi[2] = b.z; bi[3] = b.w;
  } else {
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      lo[x] = x < left ? p.lower[h * p.d + i + x] : 0.f;
      bi[x] = x < left ? p.f_bias[h * p.d + i + x] : 0.f;
    }
  }
#pragma unroll
  for (int x = 0; x < 4; ++x) {
    k[x] = 0.f;
    lf[x] = 0.f;
    if (on && x < left) {
      float sg, sn;
      ls_sigmoids(z[x] + bi[x], &sg, &sn);
      const float kk = (1.0f - lo[x]) * sn;
      // the decay's logarithm from 1 - k where k is small, so that decays close to one keep their digits; decays below
      // 2^-100 count as that
      const float ln = kk < 0.5f ? log1pf(-kk) : logf(fmaf(1.0f - lo[x], sg, lo[x]));
      k[x] = kk;
      lf[x] = fmaxf(ln * 1.4426950408889634f, -100.f);
    }
  }
}

// running sums down the columns of G [64][D + 4]; tot: [NT / D][D]
template <int D, int NT>
__device__ __forceinline__ void lsm_cumsum(float (*G)[D + 4], float (*tot)[D]) {
  constexpr int SEGS = NT / D, PER = LSM_C / SEGS;
  const int seg = threadIdx.x / D, i = threadIdx.x - seg * D;
  float run = 0.f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    run += G[seg * PER + j][i];
    G[seg * PER + j][i] = run;
  }
  tot[seg][i] = run;
  __syncthreads();
  float off = 0.f;
  for (int s = 0; s < seg; ++s) off += tot[s][i];
  if (seg > 0) {
#pragma unroll
    for (int j = 0; j < PER; ++j) G[seg * PER + j][i] += off;
  }
  __syncthreads();
}

template <int DV, int NT>
__device__ __forceinline__ void lsm_stage_v(bf16 (*dst)[DV + 8], const bf16* v, const LsArgs& p, int t0, int n, bool wide) {
#pragma unroll 4
  for (int e = threadIdx.x * 4; e < LSM_C * DV; e += NT * 4) {
    const int j = e / DV, c = e - j * DV;
    if (wide && j < n && c + 4 <= p.dv) {
      *(uint2*)&dst[j][c] = *(const uint2*)(v + (size_t)(t0 + j) * p.stride + c);
    } else {
      float o[4];
      ltc_fetch4<true>(v + (size_t)(t0 + j) * p.stride + c, j < n, false, p.dv - c, o);
      ltc_store4(&dst[j][c], o);
    }
  }
}

// ---------------------------------------------------------------------------
// pass 1
// ---------------------------------------------------------------------------
template <int D, int DV, bool GATE> struct LsmSmem1 {
  bf16 kh[LSM_C][D + 8], kl[LSM_C][D + 8], v[LSM_C][DV + 8];
  float G[GATE ? LSM_C : 1][D + 4], tot[GATE ? 256 / D : 1][D];
};

template <int D, int DV, bool GATE>
__global__ void __launch_bounds__(256, D <= 64 ? 4 : 2)
ls_mma_pass1_kernel(const bf16* a, LsArgs p, const float2* table, int wide_, float* work, float* gsum, const int* q_start,
                    int chunk0, int max_chunks) {
  extern __shared__ __align__(16) unsigned char lsm_raw[];
  LsmSmem1<D, DV, GATE>& sm = *reinterpret_cast<LsmSmem1<D, DV, GATE>*>(lsm_raw);
  pdl_wait();
  pdl_launch();
  const bool wide = wide_ != 0;
  const int h = blockIdx.x, s = blockIdx.y / max_chunks, chunk = blockIdx.y % max_chunks;
  const int t0 = q_start[s] + (chunk0 + chunk) * LSM_C;
  const int n = min(LSM_C, q_start[s + 1] - t0);
  if (n <= 0) return;
  const int hd = p.heads * p.d;
  const bf16* k = a + hd + (size_t)h * p.d;
  const bf16* v = a + 2 * (size_t)hd + (size_t)h * p.dv;
  lsm_stage_v<DV, 256>(sm.v, v, p, t0, n, wide);
  if (GATE) {
    constexpr int ITER = LSM_C * D / 1024;
    float kk[ITER][4];
#pragma unroll
    for (int u = 0; u < ITER; ++u) {
      const int e = (u * 256 + threadIdx.x) * 4, j = e / D, i = e - j * D;
      float lf[4];
      lsm_gate4(k + (size_t)(t0 + j) * p.stride + i, p, h, i, j < n, wide, kk[u], lf);
      *(float4*)&sm.G[j][i] = make_float4(lf[0], lf[1], lf[2], lf[3]);
    }
    __syncthreads();
    lsm_cumsum<D, 256>(sm.G, sm.tot);
#pragma unroll
    for (int u = 0; u < ITER; ++u) {
      const int e = (u * 256 + threadIdx.x) * 4, j = e / D, i = e - j * D;
      const float4 g = *(const float4*)&sm.G[j][i], last = *(const float4*)&sm.G[LSM_C - 1][i];
      const float w[4] = {kk[u][0] * cdm_exp2(last.x - g.x), kk[u][1] * cdm_exp2(last.y - g.y),
                          kk[u][2] * cdm_exp2(last.z - g.z), kk[u][3] * cdm_exp2(last.w - g.w)};
      lsm_split4(w, &sm.kh[j][i], &sm.kl[j][i]);
    }
    for (int i = threadIdx.x; i < p.d; i += 256) gsum[((size_t)blockIdx.y * p.heads + h) * p.d + i] = sm.G[LSM_C - 1][i];
  } else {
    const float l2 = log2f(p.decay[h]);
    lsm_rotated<D, 256, false>(a + (size_t)h * p.d, k, p, table, t0, n, wide,
        [&](int j, int col, int left, const float (&)[4], const float (&kv)[4]) {
          const float w = j < n ? ltc_pow(l2, n - 1 - j) : 0.f;
          const float kw[4] = {kv[0] * w, kv[1] * w, kv[2] * w, kv[3] * w};
          lsm_put4(sm.kh[j], sm.kl[j], col, left, kw);
        });
  }
  __syncthreads();
  // a warp owns DV / 4 value columns and half of the d rows
  constexpr int MT = D / 32, NT = DV / 32;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, c0 = (warp & 3) * (DV / 4), m0 = (warp >> 2) * (D / 2);
  float acc[MT][NT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[mt][nt][x] = 0.f;
#pragma unroll
  for (int kk = 0; kk < LSM_C; kk += 16) {
    uint32_t b[NT / 2][4];
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) ltc_b_t<DV + 8>(b[np], &sm.v[0][0], c0 + np * 16, kk);
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      uint32_t ah[4], al[4];
      ltc_a_t<D + 8>(ah, &sm.kh[0][0], m0 + mt * 16, kk);
      ltc_a_t<D + 8>(al, &sm.kl[0][0], m0 + mt * 16, kk);
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        tgm_mma(acc[mt][2 * np], ah, b[np][0], b[np][1]);
        tgm_mma(acc[mt][2 * np + 1], ah, b[np][2], b[np][3]);
        tgm_mma(acc[mt][2 * np], al, b[np][0], b[np][1]);
        tgm_mma(acc[mt][2 * np + 1], al, b[np][2], b[np][3]);
      }
    }
  }
  float* z = work + ((size_t)blockIdx.y * p.heads + h) * p.d * p.dv;
  const int g = lane >> 2, tq = lane & 3;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int c = c0 + nt * 8 + 2 * tq, i = m0 + mt * 16 + g;
      ltc_put2(z, i, c, p.d, p.dv, acc[mt][nt][0], acc[mt][nt][1]);
      ltc_put2(z, i + 8, c, p.d, p.dv, acc[mt][nt][2], acc[mt][nt][3]);
    }
}

// ---------------------------------------------------------------------------
// the chain: work[chunk] holds end states from zero; afterwards start states; the slot holds the new state
// ---------------------------------------------------------------------------
template <bool GATE, int V>
__global__ void __launch_bounds__(128)
ls_chain_kernel(LsArgs p, float* state, float* work, const float* gsum, const int* q_start, const int* slots, int num_slots,
                int chunk0, int max_chunks, int* err) {
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, s = blockIdx.y, size = p.d * p.dv;
  const int e = (blockIdx.z * blockDim.x + threadIdx.x) * V;
  if (e >= size) return;
  const int slot = slots[s], len = min(q_start[s + 1] - q_start[s] - chunk0 * LSM_C, max_chunks * LSM_C);
  if (slot < 0 || slot >= num_slots) {
    if (e == 0) atomicOr(err, 8);
    return;
  }
  if (len <= 0) return;
  const int row = e / p.dv;
  const float l2 = GATE ? 0.f : log2f(p.decay[h]);
  float* sp = state + ((size_t)slot * p.heads + h) * size + e;
  float* w0 = work + ((size_t)s * max_chunks * p.heads + h) * size + e;
  const float* g0 = GATE ? gsum + ((size_t)s * max_chunks * p.heads + h) * p.d + row : nullptr;
  const size_t step = (size_t)p.heads * size, gstep = (size_t)p.heads * p.d;
  const int chunks = (len + LSM_C - 1) / LSM_C;
  float cur[V];
  if (V == 4) { const float4 x = *(const float4*)sp; cur[0] = x.x; cur[1 % V] = x.y; cur[2 % V] = x.z; cur[3 % V] = x.w; }
  else cur[0] = sp[0];
  for (int c0 = 0; c0 < chunks; c0 += 8) {          // eight chunks' loads are on their way before the chain needs them
    float z[8][V], f[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const bool on = c0 + u < chunks;
      if (V == 4) {
        const float4 x = on ? *(const float4*)(w0 + (size_t)(c0 + u) * step) : make_float4(0.f, 0.f, 0.f, 0.f);
        z[u][0] = x.x; z[u][1 % V] = x.y; z[u][2 % V] = x.z; z[u][3 % V] = x.w;
      } else {
        z[u][0] = on ? w0[(size_t)(c0 + u) * step] : 0.f;
      }
      if (GATE) f[u] = on ? g0[(size_t)(c0 + u) * gstep] : 0.f;
    }
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (c0 + u < chunks) {
        const float keep = GATE ? exp2f(f[u]) : ltc_pow(l2, min(LSM_C, len - (c0 + u) * LSM_C));
        float* w = w0 + (size_t)(c0 + u) * step;
        if (V == 4) *(float4*)w = make_float4(cur[0], cur[1 % V], cur[2 % V], cur[3 % V]);
        else w[0] = cur[0];
#pragma unroll
        for (int x = 0; x < V; ++x) cur[x] = fmaf(keep, cur[x], z[u][x]);
      }
    }
  }
  if (V == 4) *(float4*)sp = make_float4(cur[0], cur[1 % V], cur[2 % V], cur[3 % V]);
  else sp[0] = cur[0];
}

// ---------------------------------------------------------------------------
// pass 2: 16 warps; warp w makes rows 16 (w & 3) .. of the chunk and a quarter of the value columns
// ---------------------------------------------------------------------------
#define LSM_T2 512
template <int D, bool GATE> struct LsmQ;
template <int D> struct LsmQ<D, true> { float q[LSM_C][D + 4], G[LSM_C][D + 4]; };
template <int D> struct LsmQ<D, false> { bf16 qh[LSM_C][D + 8], ql[LSM_C][D + 8]; };
template <int D, bool GATE> struct LsmK;
template <int D> struct LsmK<D, true> { float k[LSM_C][D + 4]; bf16 kh[LSM_C][D + 8], kl[LSM_C][D + 8]; };
template <int D> struct LsmK<D, false> { bf16 kh[LSM_C][D + 8], kl[LSM_C][D + 8]; };
template <int D, int DV> struct LsmS { bf16 sh[D][DV + 8], sl[D][DV + 8]; };
template <int D, int DV, bool GATE> struct LsmSmem2 {
  LsmQ<D, GATE> q;
  union { LsmK<D, GATE> k; LsmS<D, DV> s; } u;        // the keys make A, then S_0 takes their place
  bf16 v[LSM_C][DV + 8], ah[LSM_C][LSM_C + 8], al[LSM_C][LSM_C + 8];
  float ss[4][LSM_C], tot[GATE ? LSM_T2 / D : 1][D];
};

// The A fragment of rows r0 .., columns k0 .. of q * 2^(G - ref) (ref: a row of G, or null: 2^G), as value and remainder
template <int D>
__device__ __forceinline__ void lsm_decayed_a(uint32_t (&hi)[4], uint32_t (&lo)[4], const float (*q)[D + 4], const float (*G)[D + 4],
                                              const float* ref, int r0, int k0) {
  const int lane = threadIdx.x & 31, g = lane >> 2, tq = lane & 3;
#pragma unroll
  for (int x = 0; x < 4; ++x) {
    const int r = r0 + g + 8 * (x & 1), c = k0 + 2 * tq + 8 * (x >> 1);
    const float2 qv = *(const float2*)&q[r][c], gv = *(const float2*)&G[r][c];
    float2 rv = make_float2(0.f, 0.f);
    if (ref) rv = *(const float2*)&ref[c];
    cdm_split2(qv.x * cdm_exp2(gv.x - rv.x), qv.y * cdm_exp2(gv.y - rv.y), hi[x], lo[x]);
  }
}

template <int D, int DV, bool GATE>
__global__ void __launch_bounds__(LSM_T2, D <= 64 ? 2 : 1)      // (two blocks' shared memory fits an SM where D is 64)
ls_mma_pass2_kernel(const bf16* a, LsArgs p, const float2* table, int wide_, const float* work, const int* q_start,
                    int chunk0, int max_chunks, bf16* out) {
  extern __shared__ __align__(16) unsigned char lsm_raw[];
  LsmSmem2<D, DV, GATE>& sm = *reinterpret_cast<LsmSmem2<D, DV, GATE>*>(lsm_raw);
  pdl_wait();
  pdl_launch();
  const bool wide = wide_ != 0;
  const int h = blockIdx.x, s = blockIdx.y / max_chunks, chunk = blockIdx.y % max_chunks;
  const int t0 = q_start[s] + (chunk0 + chunk) * LSM_C;
  const int n = min(LSM_C, q_start[s + 1] - t0);
  if (n <= 0) return;
  const int hd = p.heads * p.d, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const bf16* q = a + (size_t)h * p.d;
  const bf16* k = q + hd;
  const bf16* v = a + 2 * (size_t)hd + (size_t)h * p.dv;
  const bf16* gate = v + (size_t)p.heads * p.dv;
  // the start state's loads are on their way while A is made; it takes the keys' place afterwards
  constexpr int SIT = D * DV / (LSM_T2 * 4);
  float s0[SIT][4];
  const float* sp = work + ((size_t)blockIdx.y * p.heads + h) * p.d * p.dv;
  const bool whole = p.d == D && p.dv == DV;
#pragma unroll
  for (int u = 0; u < SIT; ++u) {
    const int e = (u * LSM_T2 + tid) * 4, i = e / DV, c = e - i * DV;
    if (whole) {
      const float4 x = *(const float4*)(sp + e);
      s0[u][0] = x.x; s0[u][1] = x.y; s0[u][2] = x.z; s0[u][3] = x.w;
    } else {
#pragma unroll
      for (int y = 0; y < 4; ++y) s0[u][y] = (i < p.d && c + y < p.dv) ? sp[(size_t)i * p.dv + c + y] : 0.f;
    }
  }
  const float l2 = GATE ? 0.f : log2f(p.decay[h]);
  lsm_stage_v<DV, LSM_T2>(sm.v, v, p, t0, n, wide);
  if constexpr (GATE) {
    LsmK<D, true>& K = sm.u.k;
    LsmQ<D, true>& Q = sm.q;
#pragma unroll 4
    for (int e = tid * 4; e < LSM_C * D; e += LSM_T2 * 4) {
      const int j = e / D, i = e - j * D;
      const size_t at = (size_t)(t0 + j) * p.stride + i;
      float qq[4], kk[4], lf[4];
      ltc_fetch4<true>(q + at, j < n, wide, p.d - i, qq);
      lsm_gate4(k + at, p, h, i, j < n, wide, kk, lf);
      *(float4*)&Q.q[j][i] = make_float4(ls_silu(qq[0]), ls_silu(qq[1]), ls_silu(qq[2]), ls_silu(qq[3]));
      *(float4*)&K.k[j][i] = make_float4(kk[0], kk[1], kk[2], kk[3]);
      *(float4*)&Q.G[j][i] = make_float4(lf[0], lf[1], lf[2], lf[3]);
    }
    __syncthreads();
    lsm_cumsum<D, LSM_T2>(Q.G, sm.tot);
    // the keys, decayed to the end of their block of sixteen
#pragma unroll 4
    for (int e = tid * 4; e < (LSM_C - 16) * D; e += LSM_T2 * 4) {
      const int j = e / D, i = e - j * D;
      const float4 kk = *(const float4*)&K.k[j][i], gj = *(const float4*)&Q.G[j][i], ge = *(const float4*)&Q.G[j | 15][i];
      const float w[4] = {kk.x * cdm_exp2(ge.x - gj.x), kk.y * cdm_exp2(ge.y - gj.y), kk.z * cdm_exp2(ge.z - gj.z),
                          kk.w * cdm_exp2(ge.w - gj.w)};
      lsm_split4(w, &K.kh[j][i], &K.kl[j][i]);
    }
    // inside the blocks of sixteen: tiles of 2 x 2 tokens of the lower triangles (36 a block), eight slices of the channels
    for (int it = tid; it < 4 * 36 * 8; it += LSM_T2) {
      const int slice = it & 7, tile = it >> 3, b = tile / 36, w = tile - b * 36;
      int ti = (int)((sqrtf(8.0f * (float)w + 1.0f) - 1.0f) * 0.5f);
      while ((ti + 1) * (ti + 2) / 2 <= w) ++ti;
      while (ti * (ti + 1) / 2 > w) --ti;
      const int tj = w - ti * (ti + 1) / 2, r = b * 16 + ti * 2, c = b * 16 + tj * 2;
      float s00 = 0.f, s10 = 0.f, s11 = 0.f, s01 = 0.f;
#pragma unroll 4
      for (int x = slice * 2; x < D; x += 16) {
        const float2 q0 = *(const float2*)&Q.q[r][x], q1 = *(const float2*)&Q.q[r + 1][x];
        const float2 k0 = *(const float2*)&K.k[c][x], k1 = *(const float2*)&K.k[c + 1][x];
        const float2 g0 = *(const float2*)&Q.G[r][x], g1 = *(const float2*)&Q.G[r + 1][x];
        const float2 h0 = *(const float2*)&Q.G[c][x], h1 = *(const float2*)&Q.G[c + 1][x];
        s00 = fmaf(q0.x * k0.x, cdm_exp2(g0.x - h0.x), s00); s00 = fmaf(q0.y * k0.y, cdm_exp2(g0.y - h0.y), s00);
        s10 = fmaf(q1.x * k0.x, cdm_exp2(g1.x - h0.x), s10); s10 = fmaf(q1.y * k0.y, cdm_exp2(g1.y - h0.y), s10);
        s11 = fmaf(q1.x * k1.x, cdm_exp2(g1.x - h1.x), s11); s11 = fmaf(q1.y * k1.y, cdm_exp2(g1.y - h1.y), s11);
        if (ti != tj) {                         // (on the diagonal that pair looks ahead)
          s01 = fmaf(q0.x * k1.x, cdm_exp2(g0.x - h1.x), s01); s01 = fmaf(q0.y * k1.y, cdm_exp2(g0.y - h1.y), s01);
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1) {
        s00 += __shfl_xor_sync(0xffffffffu, s00, o); s01 += __shfl_xor_sync(0xffffffffu, s01, o);
        s10 += __shfl_xor_sync(0xffffffffu, s10, o); s11 += __shfl_xor_sync(0xffffffffu, s11, o);
      }
      if (slice == 0) {
        uint32_t hi, lo;
        cdm_split2(s00, s01, hi, lo);
        *(uint32_t*)&sm.ah[r][c] = hi; *(uint32_t*)&sm.al[r][c] = lo;
        cdm_split2(s10, s11, hi, lo);
        *(uint32_t*)&sm.ah[r + 1][c] = hi; *(uint32_t*)&sm.al[r + 1][c] = lo;
        if (ti != tj) {                         // the mirror image in the same block is hidden
          *(uint32_t*)&sm.ah[c][r] = 0u; *(uint32_t*)&sm.al[c][r] = 0u;
          *(uint32_t*)&sm.ah[c + 1][r] = 0u; *(uint32_t*)&sm.al[c + 1][r] = 0u;
        }
      }
    }
    __syncthreads();
  } else {
    LsmK<D, false>& K = sm.u.k;
    LsmQ<D, false>& Q = sm.q;
    lsm_rotated<D, LSM_T2, true>(q, k, p, table, t0, n, wide,
        [&](int j, int col, int left, const float (&qv)[4], const float (&kv)[4]) {
          lsm_put4(Q.qh[j], Q.ql[j], col, left, qv);
          lsm_put4(K.kh[j], K.kl[j], col, left, kv);
        });
    __syncthreads();
  }
  // A between blocks (and, with fixed decays, inside them): a warp a 16 x 16 tile
  {
    const int I = warp & 3, J = warp >> 2;
    if (GATE ? J < I : J <= I) {
      float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
      for (int kk = 0; kk < D; kk += 16) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        if constexpr (GATE) {
          lsm_decayed_a<D>(ah, al, sm.q.q, sm.q.G, &sm.q.G[J * 16 + 15][0], I * 16, kk);
        } else {
          ltc_a<D + 8>(ah, &sm.q.qh[0][0], I * 16, kk);
          ltc_a<D + 8>(al, &sm.q.ql[0][0], I * 16, kk);
        }
        ltc_b<D + 8>(bh, &sm.u.k.kh[0][0], J * 16, kk);
        ltc_b<D + 8>(bl, &sm.u.k.kl[0][0], J * 16, kk);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          tgm_mma(acc[x], ah, bh[2 * x], bh[2 * x + 1]);
          tgm_mma(acc[x], ah, bl[2 * x], bl[2 * x + 1]);
          tgm_mma(acc[x], al, bh[2 * x], bh[2 * x + 1]);
        }
      }
#pragma unroll
      for (int x = 0; x < 2; ++x)
#pragma unroll
        for (int y = 0; y < 2; ++y) {
          const int t = I * 16 + g + 8 * y, j = J * 16 + x * 8 + 2 * tq;
          float f0 = acc[x][2 * y], f1 = acc[x][2 * y + 1];
          if (!GATE) {
            f0 = j <= t ? f0 * ltc_pow(l2, t - j) : 0.f;
            f1 = j + 1 <= t ? f1 * ltc_pow(l2, t - j - 1) : 0.f;
          }
          uint32_t hi, lo;
          cdm_split2(f0, f1, hi, lo);
          *(uint32_t*)&sm.ah[t][j] = hi;
          *(uint32_t*)&sm.al[t][j] = lo;
        }
    }
  }
  __syncthreads();
#pragma unroll
  for (int u = 0; u < SIT; ++u) {
    const int e = (u * LSM_T2 + tid) * 4, i = e / DV, c = e - i * DV;
    lsm_split4(s0[u], &sm.u.s.sh[i][c], &sm.u.s.sl[i][c]);
  }
  __syncthreads();
  constexpr int NT = DV / 32;                     // n-tiles a warp
  const int r0 = (warp & 3) * 16, cbase = (warp >> 2) * (DV / 4);
  float o[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; ++nt)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[nt][x] = 0.f;
#pragma unroll
  for (int kk = 0; kk < D; kk += 16) {
    uint32_t ah[4], al[4];
    if constexpr (GATE) {
      lsm_decayed_a<D>(ah, al, sm.q.q, sm.q.G, nullptr, r0, kk);
    } else {
      ltc_a<D + 8>(ah, &sm.q.qh[0][0], r0, kk);
      ltc_a<D + 8>(al, &sm.q.ql[0][0], r0, kk);
    }
#pragma unroll
    for (int np = 0; np < NT / 2; ++np) {
      uint32_t bh[4], bl[4];
      ltc_b_t<DV + 8>(bh, &sm.u.s.sh[0][0], cbase + np * 16, kk);
      ltc_b_t<DV + 8>(bl, &sm.u.s.sl[0][0], cbase + np * 16, kk);
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        tgm_mma(o[2 * np + x], ah, bh[2 * x], bh[2 * x + 1]);
        tgm_mma(o[2 * np + x], ah, bl[2 * x], bl[2 * x + 1]);
        tgm_mma(o[2 * np + x], al, bh[2 * x], bh[2 * x + 1]);
      }
    }
  }
  if (!GATE) {
    const float up = ltc_pow(l2, r0 + g + 1), dn = ltc_pow(l2, r0 + g + 9);
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) { o[nt][0] *= up; o[nt][1] *= up; o[nt][2] *= dn; o[nt][3] *= dn; }
  }
#pragma unroll
  for (int ks = 0; ks < LSM_C / 16; ++ks) {
    if (ks * 16 <= r0) {
      uint32_t ah[4], al[4];
      ltc_a<LSM_C + 8>(ah, &sm.ah[0][0], r0, ks * 16);
      ltc_a<LSM_C + 8>(al, &sm.al[0][0], r0, ks * 16);
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t b[4];
        ltc_b_t<DV + 8>(b, &sm.v[0][0], cbase + np * 16, ks * 16);
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          tgm_mma(o[2 * np + x], ah, b[2 * x], b[2 * x + 1]);
          tgm_mma(o[2 * np + x], al, b[2 * x], b[2 * x + 1]);
        }
      }
    }
  }
  // a row's sum of squares: over the quad, then over the four warps that share the row
  float ss[2] = {0.f, 0.f};
#pragma unroll
  for (int nt = 0; nt < NT; ++nt) {
    ss[0] = fmaf(o[nt][0], o[nt][0], fmaf(o[nt][1], o[nt][1], ss[0]));
    ss[1] = fmaf(o[nt][2], o[nt][2], fmaf(o[nt][3], o[nt][3], ss[1]));
  }
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    ss[y] += __shfl_xor_sync(0xffffffffu, ss[y], 1);
    ss[y] += __shfl_xor_sync(0xffffffffu, ss[y], 2);
    if (tq == 0) sm.ss[warp >> 2][r0 + g + 8 * y] = ss[y];
  }
  __syncthreads();
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    const int t = r0 + g + 8 * y;
    if (t >= n) continue;
    const float rr = 1.0f / sqrtf((sm.ss[0][t] + sm.ss[1][t] + sm.ss[2][t] + sm.ss[3][t]) / (float)p.dv + p.eps);
    const bf16* gr = gate + (size_t)(t0 + t) * p.stride;
    bf16* orow = out + ((size_t)(t0 + t) * p.heads + h) * p.dv;
    const bool pair = (p.dv & 1) == 0 && (p.stride & 1) == 0;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) {
      const int c = cbase + nt * 8 + 2 * tq;
      float y0 = o[nt][2 * y] * rr, y1 = o[nt][2 * y + 1] * rr;
      if (pair && wide && c + 1 < p.dv) {
        if (p.norm_w) { y0 *= p.norm_w[c]; y1 *= p.norm_w[c + 1]; }
        if (p.gated) {
          const float2 gv = __bfloat1622float2(*(const __nv_bfloat162*)(gr + c));
          y0 *= ls_silu(gv.x);
          y1 *= ls_silu(gv.y);
        }
        *(__nv_bfloat162*)(orow + c) = __floats2bfloat162_rn(y0, y1);
      } else {
        if (c < p.dv) {
          if (p.norm_w) y0 *= p.norm_w[c];
          if (p.gated) y0 *= ls_silu(__bfloat162float(gr[c]));
          orow[c] = __float2bfloat16_rn(y0);
        }
        if (c + 1 < p.dv) {
          if (p.norm_w) y1 *= p.norm_w[c + 1];
          if (p.gated) y1 *= ls_silu(__bfloat162float(gr[c + 1]));
          orow[c + 1] = __float2bfloat16_rn(y1);
        }
      }
    }
  }
}

template <int D, int DV, bool GATE>
static int lsm_launch(const bf16* a, LsArgs p, const float2* table, float* state, float* work, float* gsum, const int* q_start,
                      const int* slots, int num_slots, int num_seqs, int chunk0, int max_chunks, bf16* out, int* err,
                      cudaStream_t stream) {
  const size_t s1 = sizeof(LsmSmem1<D, DV, GATE>), s2 = sizeof(LsmSmem2<D, DV, GATE>);
  static bool allowed = false;
  if (!allowed) {
    cudaError_t e = cudaFuncSetAttribute(ls_mma_pass1_kernel<D, DV, GATE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(ls_mma_pass2_kernel<D, DV, GATE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s2);
    if (e != cudaSuccess) return (int)e;
    allowed = true;
  }
  // rows that start on 8-byte boundaries are fetched four values a load (the rotated pairs' partners too)
  const int wide = p.stride % 4 == 0 && p.d % 4 == 0 && p.dv % 4 == 0 && p.rd % 8 == 0 && (((uintptr_t)a) & 7) == 0 &&
                   (((uintptr_t)p.lower | (uintptr_t)p.f_bias) & 15) == 0;
  const dim3 grid(p.heads, num_seqs * max_chunks);
  rllm_launch_pdl(ls_mma_pass1_kernel<D, DV, GATE>, grid, dim3(256), s1, stream, a, p, table, wide, work, gsum, q_start,
                  chunk0, max_chunks);
  if (p.dv % 4 == 0)
    rllm_launch_pdl(ls_chain_kernel<GATE, 4>, dim3(p.heads, num_seqs, (p.d * p.dv / 4 + 127) / 128), dim3(128), (size_t)0, stream,
                    p, state, work, (const float*)gsum, q_start, slots, num_slots, chunk0, max_chunks, err);
  else
    rllm_launch_pdl(ls_chain_kernel<GATE, 1>, dim3(p.heads, num_seqs, (p.d * p.dv + 127) / 128), dim3(128), (size_t)0, stream, p,
                    state, work, (const float*)gsum, q_start, slots, num_slots, chunk0, max_chunks, err);
  rllm_launch_pdl(ls_mma_pass2_kernel<D, DV, GATE>, grid, dim3(LSM_T2), s2, stream, a, p, table, wide, (const float*)work, q_start,
                  chunk0, max_chunks, out);
  return 0;
}
