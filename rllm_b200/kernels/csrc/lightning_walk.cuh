// The walk of the linear-attention recurrence  S_t = lambda S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t  on the
// CUDA cores, in two forms that share every line but the token's factors:
//   STEPS false   lambda is one number per head, and q, k, v are activated (silu) as they are read
//                 (lightning attention; see lightning.cu)
//   STEPS true    lambda and a factor on k come from a step size per head and token, q and k are shared by
//                 the heads of a group, nothing is activated, and d_h v_t is added to the result
//                 (the state-space recurrence; see ssd.cu)
// What a block and a thread do is told in lightning.cu.
#pragma once
#include "common.cuh"
#include <math.h>

// what the recurrence with step sizes reads besides q, k and v
struct LtSteps {
  const float* dt;           // [T, heads]: the steps before bias and softplus
  const float* dt_bias;      // [heads]
  const float* a_log;        // [heads]: lambda_t = exp(-exp(a_log) dt_t)
  const float* skip;         // [heads]: d_h
  float* chunk_dt;           // [chunks, heads]: the sum of a chunk's step sizes
  int per;                   // heads that share a group's q and k
};
__device__ __forceinline__ float lt_step(const LtSteps& p, int t, int h, int heads) {
  const float v = p.dt[(size_t)t * heads + h] + p.dt_bias[h];
  return v > 20.f ? v : log1pf(expf(v));
}

#define LT_TOKENS 8
#define LT_CHUNK 64
#define LT_TILE 8            // a thread's tile of S is LT_TILE x LT_TILE
#define LT_MAX_COLS 256      // value columns a block covers at most

__device__ __forceinline__ float lt_silu(float v) { return v / (1.0f + expf(-v)); }
template <bool STEPS> __device__ __forceinline__ float lt_act(float v) { return STEPS ? v : lt_silu(v); }

// mode 0: whole portion from the slot's state, state written back
// mode 1: one chunk from a zero start, end state to work[chunk], no output
// mode 2: one chunk from work[chunk], output, nothing written back
// NS: slices of d (a power of two up to 32; d <= 8 NS); thread = slice + NS * (tile of columns)
template <typename T, int NS, int MODE, bool STEPS>
__global__ void __launch_bounds__(256)
lightning_kernel(const T* q, const T* k, const T* v, int stride, const float* decay, LtSteps steps, float* state,
                 float* work, const int* q_start, const int* slots, int num_slots, int max_chunks, float* out,
                 int heads, int d, int dv, int* err) {
  constexpr int D = NS * LT_TILE;
  __shared__ __align__(16) float qs[LT_TOKENS][D], ks[LT_TOKENS][D], vs[LT_TOKENS][LT_MAX_COLS];
  __shared__ float keep_s[LT_TOKENS], take_s[LT_TOKENS];
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x;
  const int s = (MODE == 0) ? blockIdx.y : blockIdx.y / max_chunks;
  const int chunk = (MODE == 0) ? 0 : blockIdx.y % max_chunks;
  const int cols = (int)blockDim.x / NS * LT_TILE;              // value columns of this block
  const int col0 = blockIdx.z * cols;
  const int ds = threadIdx.x % NS, vt = threadIdx.x / NS;
  const int i0 = ds * LT_TILE, jl = vt * LT_TILE, j0 = col0 + jl;
  int t0 = q_start[s], t1 = q_start[s + 1];
  if (MODE != 0) {
    t0 += chunk * LT_CHUNK;
    t1 = min(t1, t0 + LT_CHUNK);
    if (t0 >= t1) return;
  }
  const int slot = slots[s];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, 8);
    return;
  }
  float lam = 0.f, rate = 0.f, skip = 0.f, dt_sum = 0.f;
  if (STEPS) { rate = expf(steps.a_log[h]); skip = steps.skip[h]; } else { lam = decay[h]; }
  const int hk = STEPS ? h / steps.per : h;                     // whose q and k this head reads
  // which finished output columns this lane holds after the sum over the slices (see below)
  int colbase = 0, last = LT_TILE;
  bool writer = true;
#pragma unroll
  for (int off = NS / 2; off > 0; off >>= 1) {
    const bool upper = (ds & off) != 0;
    if (last > 1) {
      last >>= 1;
      colbase += upper ? last : 0;
    } else {
      writer = writer && !upper;
    }
  }
  float S[LT_TILE][LT_TILE];
  float* sp = (MODE == 0) ? state + ((size_t)slot * heads + h) * d * dv
                          : work + ((size_t)blockIdx.y * heads + h) * d * dv;
  // a tile's rows are eight consecutive floats: two 16-byte accesses where the head's sizes allow it
  const bool wide = (dv & 3) == 0 && j0 + LT_TILE <= dv && (((uintptr_t)sp) & 15) == 0;
#pragma unroll
  for (int a = 0; a < LT_TILE; ++a) {
    if (MODE != 1 && wide && i0 + a < d) {
      *(float4*)&S[a][0] = *(const float4*)(sp + (size_t)(i0 + a) * dv + j0);
      *(float4*)&S[a][4] = *(const float4*)(sp + (size_t)(i0 + a) * dv + j0 + 4);
    } else {
#pragma unroll
      for (int b = 0; b < LT_TILE; ++b)
        S[a][b] = (MODE != 1 && i0 + a < d && j0 + b < dv) ? sp[(size_t)(i0 + a) * dv + j0 + b] : 0.f;
    }
  }
  // The next eight tokens' rows are fetched into registers before this eight's arithmetic starts, so that the
  // loads' latency lies behind it (with four slices or more: a thread then stages at most 8 + 8 + 16 values).
  constexpr bool PF = NS >= 4;
  constexpr int PQ = 8, PV = PF ? 64 / NS : 1;
  T rq[PQ], rk[PQ], rv[PV];
  auto fetch = [&](int tb) {
    const int n = min(LT_TOKENS, t1 - tb);
#pragma unroll
    for (int u = 0; u < PQ; ++u) {
      const int e = threadIdx.x + u * blockDim.x;
      const int tt = e / D, i = e - tt * D;
      const bool on = e < LT_TOKENS * D && tt < n && i < d;
      const size_t at = (size_t)(tb + tt) * stride + (size_t)hk * d + i;
      rq[u] = (on && MODE != 1) ? q[at] : from_f32<T>(0.f);
      rk[u] = on ? k[at] : from_f32<T>(0.f);
    }
#pragma unroll
    for (int u = 0; u < PV; ++u) {
      const int e = threadIdx.x + u * blockDim.x;
      const int tt = e / cols, j = e - tt * cols;
      const bool on = e < LT_TOKENS * cols && tt < n && col0 + j < dv;
      rv[u] = on ? v[(size_t)(tb + tt) * stride + (size_t)h * dv + col0 + j] : from_f32<T>(0.f);
    }
  };
  if (PF) fetch(t0);
  for (int tb = t0; tb < t1; tb += LT_TOKENS) {
    const int n = min(LT_TOKENS, t1 - tb);
    __syncthreads();
    if (PF) {
#pragma unroll
      for (int u = 0; u < PQ; ++u) {
        const int e = threadIdx.x + u * blockDim.x;
        if (e < LT_TOKENS * D) {
          (&qs[0][0])[e] = lt_act<STEPS>(to_f32(rq[u]));                 // silu(0) = 0 where nothing was fetched
          (&ks[0][0])[e] = lt_act<STEPS>(to_f32(rk[u]));
        }
      }
#pragma unroll
      for (int u = 0; u < PV; ++u) {
        const int e = threadIdx.x + u * blockDim.x;
        if (e < LT_TOKENS * cols) vs[e / cols][e % cols] = lt_act<STEPS>(to_f32(rv[u]));
      }
    } else {
      for (int e = threadIdx.x; e < LT_TOKENS * D; e += blockDim.x) {
        const int tt = e / D, i = e - tt * D;
        float qv = 0.f, kv = 0.f;
        if (tt < n && i < d) {
          const size_t at = (size_t)(tb + tt) * stride + (size_t)hk * d + i;
          if (MODE != 1) qv = lt_act<STEPS>(to_f32(q[at]));
          kv = lt_act<STEPS>(to_f32(k[at]));
        }
        qs[tt][i] = qv;
        ks[tt][i] = kv;
      }
      for (int e = threadIdx.x; e < LT_TOKENS * cols; e += blockDim.x) {
        const int tt = e / cols, j = e - tt * cols;
        vs[tt][j] = (tt < n && col0 + j < dv) ? lt_act<STEPS>(to_f32(v[(size_t)(tb + tt) * stride + (size_t)h * dv + col0 + j])) : 0.f;
      }
    }
    if (STEPS && threadIdx.x < n) {
      const float dt = lt_step(steps, tb + threadIdx.x, h, heads);
      keep_s[threadIdx.x] = expf(-rate * dt);
      take_s[threadIdx.x] = dt;
    }
    __syncthreads();
    if (PF && tb + LT_TOKENS < t1) fetch(tb + LT_TOKENS);
    for (int tt = 0; tt < n; ++tt) {
      float take = 1.f;
      if (STEPS) { lam = keep_s[tt]; take = take_s[tt]; dt_sum += take; }
      float kk[LT_TILE], qq[LT_TILE], vv[LT_TILE], o[LT_TILE];
      *(float4*)&kk[0] = *(const float4*)&ks[tt][i0];
      *(float4*)&kk[4] = *(const float4*)&ks[tt][i0 + 4];
      *(float4*)&vv[0] = *(const float4*)&vs[tt][jl];
      *(float4*)&vv[4] = *(const float4*)&vs[tt][jl + 4];
      if (MODE != 1) {
        *(float4*)&qq[0] = *(const float4*)&qs[tt][i0];
        *(float4*)&qq[4] = *(const float4*)&qs[tt][i0 + 4];
      }
#pragma unroll
      for (int b = 0; b < LT_TILE; ++b) { o[b] = 0.f; if (STEPS) vv[b] *= take; }
#pragma unroll
      for (int a = 0; a < LT_TILE; ++a)
#pragma unroll
        for (int b = 0; b < LT_TILE; ++b) {
          S[a][b] = fmaf(lam, S[a][b], kk[a] * vv[b]);
          if (MODE != 1) o[b] = fmaf(S[a][b], qq[a], o[b]);
        }
      if (MODE != 1) {
        // The sum over the slices by halving: in every round a lane hands half of its partial sums to its
        // partner and adds the partner's for the half it keeps (8 shuffles for 16 slices instead of 32);
        // at the end a lane holds the finished sums of `last` columns from `colbase` on.
        int cnt = LT_TILE;
#pragma unroll
        for (int off = NS / 2; off > 0; off >>= 1) {
          const bool upper = (ds & off) != 0;
          if (cnt > 1) {
            cnt >>= 1;
#pragma unroll
            for (int b = 0; b < LT_TILE / 2; ++b) {
              if (b < cnt) {
                const float send = upper ? o[b] : o[b + cnt];
                const float recv = __shfl_xor_sync(0xffffffffu, send, off);
                o[b] = (upper ? o[b + cnt] : o[b]) + recv;
              }
            }
          } else {
            o[0] += __shfl_xor_sync(0xffffffffu, o[0], off);
          }
        }
        if (writer) {
          float* op = out + ((size_t)(tb + tt) * heads + h) * dv + j0 + colbase;
#pragma unroll
          for (int b = 0; b < LT_TILE; ++b)
            if (b < last && j0 + colbase + b < dv) op[b] = STEPS ? fmaf(skip, vs[tt][jl + colbase + b], o[b]) : o[b];
        }
      }
    }
  }
  if (STEPS && MODE == 1 && threadIdx.x == 0 && blockIdx.z == 0) steps.chunk_dt[(size_t)blockIdx.y * heads + h] = dt_sum;
  if (MODE != 2) {
#pragma unroll
    for (int a = 0; a < LT_TILE; ++a) {
      if (wide && i0 + a < d) {
        *(float4*)(sp + (size_t)(i0 + a) * dv + j0) = *(const float4*)&S[a][0];
        *(float4*)(sp + (size_t)(i0 + a) * dv + j0 + 4) = *(const float4*)&S[a][4];
      } else {
#pragma unroll
        for (int b = 0; b < LT_TILE; ++b)
          if (i0 + a < d && j0 + b < dv) sp[(size_t)(i0 + a) * dv + j0 + b] = S[a][b];
      }
    }
  }
}

// work[s * max_chunks + c] holds chunk c's end state from a zero start; afterwards it holds chunk c's start
// state, and the slot holds the sequence's state after its last token.
template <bool STEPS>
__global__ void __launch_bounds__(256)
lightning_chain_kernel(const float* decay, LtSteps steps, float* state, float* work, const int* q_start, const int* slots,
                       int num_slots, int max_chunks, int heads, int d, int dv) {
  pdl_wait();
  pdl_launch();
  const int h = blockIdx.x, s = blockIdx.y;
  const int e = blockIdx.z * blockDim.x + threadIdx.x;
  if (e >= d * dv) return;
  const int slot = slots[s];
  if (slot < 0 || slot >= num_slots) return;
  const int len = q_start[s + 1] - q_start[s];
  if (len <= 0) return;
  const float lam = STEPS ? 0.f : decay[h];
  const float full = STEPS ? 0.f : powf(lam, (float)LT_CHUNK);
  const float rate = STEPS ? expf(steps.a_log[h]) : 0.f;
  float* sp = state + ((size_t)slot * heads + h) * d * dv + e;
  float cur = *sp;
  const int chunks = (len + LT_CHUNK - 1) / LT_CHUNK;
  float* w0 = work + ((size_t)s * max_chunks * heads + h) * d * dv + e;
  const size_t step = (size_t)heads * d * dv;
  // eight chunks' end states are fetched before the chain runs over them (the loads do not depend on it)
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float z[8], sum[8];
#pragma unroll
    for (int u = 0; u < 8; ++u)
      sum[u] = (STEPS && c0 + u < chunks) ? steps.chunk_dt[((size_t)s * max_chunks + c0 + u) * heads + h] : 0.f;
#pragma unroll
    for (int u = 0; u < 8; ++u) z[u] = (c0 + u < chunks) ? w0[(size_t)(c0 + u) * step] : 0.f;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      if (c0 + u < chunks) {
        w0[(size_t)(c0 + u) * step] = cur;
        const int n = min(LT_CHUNK, len - (c0 + u) * LT_CHUNK);
        cur = fmaf(STEPS ? expf(-rate * sum[u]) : (n == LT_CHUNK ? full : powf(lam, (float)n)), cur, z[u]);
      }
    }
  }
  *sp = cur;
}

template <typename T, int NS, bool STEPS>
static int lightning_launch(const T* q, const T* k, const T* v, int stride, const float* decay, LtSteps steps, float* state,
                            float* work, const int* q_start, const int* slots, int num_slots, int num_seqs,
                            int max_chunks, float* out, int heads, int d, int dv, int* err, cudaStream_t stream) {
  // tiles of eight value columns a block: as many as the head has, up to 256 threads and LT_MAX_COLS columns,
  // and whole warps (a slice's partners in the sum are lanes of one warp)
  int vt = (dv + LT_TILE - 1) / LT_TILE;
  vt = vt > 8 ? vt : 8;                          // at least as many threads as a row of q has values (8 NS)
  vt = vt < 256 / NS ? vt : 256 / NS;
  vt = vt < LT_MAX_COLS / LT_TILE ? vt : LT_MAX_COLS / LT_TILE;
  while ((vt * NS) % 32) ++vt;
  const unsigned threads = (unsigned)(vt * NS), gz = (unsigned)((dv + vt * LT_TILE - 1) / (vt * LT_TILE));
  if (max_chunks <= 0) {
    rllm_launch_pdl(lightning_kernel<T, NS, 0, STEPS>, dim3(heads, num_seqs, gz), dim3(threads), (size_t)0, stream, q, k, v,
                    stride, decay, steps, state, work, q_start, slots, num_slots, 1, out, heads, d, dv, err);
  } else {
    const dim3 grid(heads, num_seqs * max_chunks, gz);
    rllm_launch_pdl(lightning_kernel<T, NS, 1, STEPS>, grid, dim3(threads), (size_t)0, stream, q, k, v, stride, decay, steps,
                    state, work, q_start, slots, num_slots, max_chunks, out, heads, d, dv, err);
    rllm_launch_pdl(lightning_chain_kernel<STEPS>, dim3(heads, num_seqs, (d * dv + 255) / 256), dim3(256), (size_t)0, stream,
                    decay, steps, state, work, q_start, slots, num_slots, max_chunks, heads, d, dv);
    rllm_launch_pdl(lightning_kernel<T, NS, 2, STEPS>, grid, dim3(threads), (size_t)0, stream, q, k, v, stride, decay, steps,
                    state, work, q_start, slots, num_slots, max_chunks, out, heads, d, dv, err);
  }
  return 0;
}

// The walk for any head: NS slices of d by its size.
template <typename T, bool STEPS>
static int lightning_walk(const T* q, const T* k, const T* v, int stride, const float* decay, LtSteps steps, float* state,
                          float* work, const int* q_start, const int* slots, int num_slots, int num_seqs,
                          int max_chunks, float* out, int heads, int d, int dv, int* err, cudaStream_t stream) {
#define LT_GO(NS_)                                                                                              \
  return lightning_launch<T, NS_, STEPS>(q, k, v, stride, decay, steps, state, work, q_start, slots, num_slots,  \
                                         num_seqs, max_chunks, out, heads, d, dv, err, stream)
  if (d <= 8) LT_GO(1);
  if (d <= 16) LT_GO(2);
  if (d <= 32) LT_GO(4);
  if (d <= 64) LT_GO(8);
  if (d <= 128) LT_GO(16);
  LT_GO(32);
#undef LT_GO
}
