// Linear attention with a matrix state per head and request:
//
//   S_t = diag(f_t) S_(t-1) + k_t v_t^T   [d, dv],     o_t = S_t^T q_t
//   y_t = o_t / sqrt(mean(o_t^2) + eps) (* w) (* silu(g_t))                  per head
//
// from a token's row of projections [q | k or f | v | (g)], in two kinds:
//
//   fixed decays ("retention")       f is one number a head; q and k are rotated by the token's position (dimension i
//                                    with i + rd / 2 over the first rd), then k is multiplied by k_scale
//   decays per channel ("hgrn2")     q <- silu(q); f = l + (1 - l) sigmoid(f + bias) with a lower bound l per channel;
//                                    k = 1 - f, taken as (1 - l) sigmoid(-(f + bias)), so that it keeps its digits
//                                    where f is close to one
//
// S lives in float32 in the request's state slot [heads][d][dv], starts at zero and is carried from step to step.
// Everything between the projections and y is float32.
//
// The walk (this file): a block owns a head of a sequence, S in registers (a thread: one or four value columns of
// every RG-th row).  Eight tokens' factors are made at a time in shared memory; a token's outputs are the sums over
// the row groups, which one warp (the warps take turns) adds up, normalises, gates and stores while the others go on.
// It serves single decoded tokens, short portions and float32; long bfloat16 portions go as chunks of 64 on the
// tensor cores (linear_state_mma.cuh).
#include "linear_state_mma.cuh"

#define LS_SEG 8

template <typename T, bool GATE, int V, int NR>
__global__ void __launch_bounds__(512)
ls_walk_kernel(const T* a, LsArgs p, float* state, const int* q_start, const int* slots, int num_slots, int cols, T* out,
               float* raw, int early, int* err) {
  extern __shared__ __align__(16) float ls_smem[];
  const int d = p.d, dv = p.dv;
  const int CG = (cols + V - 1) / V, RG = min((int)blockDim.x / CG, d);
  float* qs = ls_smem;                            // [SEG][d]
  float* ks = qs + LS_SEG * d;                    // [SEG][d]
  float* fs = ks + LS_SEG * d;                    // [SEG][d] (decays per channel)
  float* vs = fs + (GATE ? LS_SEG * d : 0);       // [SEG][CG * V]
  float* red = vs + LS_SEG * CG * V;              // [2][RG][CG * V]
  if (!early) pdl_wait();
  const int h = blockIdx.x, s = blockIdx.y, col0 = blockIdx.z * cols;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5;
  const int rg = tid / CG, cg = tid - rg * CG;
  const bool act = rg < RG;
  const int t0 = q_start[s], t1 = q_start[s + 1];
  const int slot = slots[s];
  const bool bad = slot < 0 || slot >= num_slots;
  const int cbase = col0 + cg * V;                // this thread's value columns
  float S[NR][V];
  float* sp = state + ((size_t)(bad ? 0 : slot) * p.heads + h) * d * dv + cbase;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + i * RG;
    const bool on = act && !bad && r < d && cbase < dv;
    if (V == 4) {
      const float4 x = on ? *(const float4*)(sp + (size_t)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i][0] = x.x; S[i][1 % V] = x.y; S[i][2 % V] = x.z; S[i][3 % V] = x.w;
    } else {
      S[i][0] = on ? sp[(size_t)r * dv] : 0.f;
    }
  }
  if (early) pdl_wait();
  pdl_launch();
  if (bad) {
    if (tid == 0) atomicOr(err, 8);
    return;
  }
  const int hd = p.heads * d;
  const T* aq = a + (size_t)h * d;
  const T* ak = aq + hd;
  const T* av = a + 2 * (size_t)hd + (size_t)h * dv;
  const T* ag = av + (size_t)p.heads * dv;
  const float lam = GATE ? 0.f : p.decay[h];
  for (int tb = t0; tb < t1; tb += LS_SEG) {
    const int n = min(LS_SEG, t1 - tb);
    if (GATE) {
      for (int e = tid; e < n * d; e += blockDim.x) {
        const int tt = e / d, i = e - tt * d;
        const size_t at = (size_t)(tb + tt) * p.stride + i;
        const float l = p.lower[h * d + i], z = to_f32(ak[at]) + p.f_bias[h * d + i];
        qs[e] = ls_silu(to_f32(aq[at]));
        float on, off;
        ls_sigmoids(z, &on, &off);
        fs[e] = fmaf(1.0f - l, on, l);
        ks[e] = (1.0f - l) * off;
      }
    } else {
      const int half = p.rd >> 1, items = d - half;
      for (int e = tid; e < n * items; e += blockDim.x) {
        const int tt = e / items, i = e - tt * items;
        const size_t at = (size_t)(tb + tt) * p.stride;
        if (i < half) {
          float c, sn;
          ls_cos_sin<T>(p.positions[tb + tt], p.inv_freq[i], &c, &sn);
          const float qa = to_f32(aq[at + i]), qb = to_f32(aq[at + i + half]);
          const float ka = to_f32(ak[at + i]), kb = to_f32(ak[at + i + half]);
          qs[tt * d + i] = qa * c - qb * sn;
          qs[tt * d + i + half] = qb * c + qa * sn;
          ks[tt * d + i] = (ka * c - kb * sn) * p.k_scale;
          ks[tt * d + i + half] = (kb * c + ka * sn) * p.k_scale;
        } else {
          const int j = i + half;                 // rd .. d - 1: not rotated
          qs[tt * d + j] = to_f32(aq[at + j]);
          ks[tt * d + j] = to_f32(ak[at + j]) * p.k_scale;
        }
      }
    }
    for (int e = tid; e < n * CG * V; e += blockDim.x) {
      const int tt = e / (CG * V), c = e - tt * (CG * V);
      vs[e] = (c < cols && col0 + c < dv) ? to_f32(av[(size_t)(tb + tt) * p.stride + col0 + c]) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      float* r0 = red + (tt & 1) * RG * CG * V;
      if (act) {
        float o[V], vv[V];
#pragma unroll
        for (int x = 0; x < V; ++x) { o[x] = 0.f; vv[x] = vs[tt * CG * V + cg * V + x]; }
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int r = rg + i * RG;
          if (r < d) {
            const float kk = ks[tt * d + r], qq = qs[tt * d + r], ff = GATE ? fs[tt * d + r] : lam;
#pragma unroll
            for (int x = 0; x < V; ++x) {
              S[i][x] = fmaf(ff, S[i][x], kk * vv[x]);
              o[x] = fmaf(S[i][x], qq, o[x]);
            }
          }
        }
#pragma unroll
        for (int x = 0; x < V; ++x) r0[(size_t)rg * CG * V + cg * V + x] = o[x];
      }
      __syncthreads();
      if (warp == tt % nwarps) {                  // this warp finishes the token; the others go on
        float y[8], ss = 0.f;
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const int c = lane + 32 * u;
          y[u] = 0.f;
          if (c < cols && col0 + c < dv) {
            for (int g = 0; g < RG; ++g) y[u] += r0[(size_t)g * CG * V + c];
          }
          ss = fmaf(y[u], y[u], ss);
        }
        const size_t row = (size_t)(tb + tt) * p.heads * dv + (size_t)h * dv + col0;
        if (raw) {
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const int c = lane + 32 * u;
            if (c < cols && col0 + c < dv) raw[row + c] = y[u];
          }
        } else {
          const float rr = 1.0f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
#pragma unroll
          for (int u = 0; u < 8; ++u) {
            const int c = lane + 32 * u;
            if (c < dv) {
              float v = y[u] * rr;
              if (p.norm_w) v *= p.norm_w[c];
              if (p.gated) v *= ls_silu(to_f32(ag[(size_t)(tb + tt) * p.stride + c]));
              out[row + c] = from_f32<T>(v);
            }
          }
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + i * RG;
    if (act && r < d && cbase < dv) {
      if (V == 4) *(float4*)(sp + (size_t)r * dv) = make_float4(S[i][0], S[i][1 % V], S[i][2 % V], S[i][3 % V]);
      else sp[(size_t)r * dv] = S[i][0];
    }
  }
}

// y from the sums o (heads whose columns are shared out among blocks): a warp a (token, head)
template <typename T>
__global__ void __launch_bounds__(128)
ls_norm_kernel(const float* raw, const T* a, LsArgs p, T* out, int T_tokens) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (w >= (long long)T_tokens * p.heads) return;
  const int t = (int)(w / p.heads), h = (int)(w - (long long)t * p.heads);
  const float* o = raw + (size_t)w * p.dv;
  const T* g = a + (size_t)t * p.stride + (size_t)p.heads * (2 * p.d + p.dv) + (size_t)h * p.dv;
  float ss = 0.f;
  for (int c = lane; c < p.dv; c += 32) ss = fmaf(o[c], o[c], ss);
  const float rr = 1.0f / sqrtf(warp_sum(ss) / (float)p.dv + p.eps);
  for (int c = lane; c < p.dv; c += 32) {
    float v = o[c] * rr;
    if (p.norm_w) v *= p.norm_w[c];
    if (p.gated) v *= ls_silu(to_f32(g[c]));
    out[(size_t)w * p.dv + c] = from_f32<T>(v);
  }
}

struct LsShape { int cols, threads, nr; };
// how a block of the walk covers a head: all its columns if they fit, else 64 or 32 at a time; nr 0: no form takes it
static LsShape ls_shape(int d, int dv) {
  const int V = dv % 4 == 0 ? 4 : 1, max_nr = V == 4 ? 16 : 32;
  for (int part = 0; part < 3; ++part) {
    const int cols = part == 0 ? dv : (part == 1 ? 64 : 32);
    if (cols > dv || cols > 256) continue;
    for (int threads = part == 0 ? 256 : 512; threads <= 512; threads *= 2) {
      const int cg = (cols + V - 1) / V;
      int rg = threads / cg;
      rg = rg < d ? rg : d;
      if (rg < 1) continue;
      const int nr = (d + rg - 1) / rg;
      if (nr <= max_nr) return {cols, threads, nr};
    }
  }
  return {0, 0, 0};
}

// 1: the walk leaves the sums o in `raw` ([T, heads * dv] float32, the caller's) and a second kernel makes y
RLLM_EXPORT int rllm_linear_state_needs_raw(int d, int dv) {
  const LsShape sh = ls_shape(d, dv);
  return sh.nr > 0 && sh.cols < dv ? 1 : 0;
}

template <typename T, bool GATE>
static int ls_walk(const T* a, LsArgs p, float* state, const int* q_start, const int* slots, int num_slots, int num_seqs,
                   int T_tokens, T* out, float* raw, int early, int* err, cudaStream_t stream) {
  const LsShape sh = ls_shape(p.d, p.dv);
  if (sh.nr == 0) return RLLM_E_UNSUPPORTED;
  const int gz = (p.dv + sh.cols - 1) / sh.cols;
  if (gz > 1 && !raw) return RLLM_E_BADARG;
  const int V = p.dv % 4 == 0 ? 4 : 1, cg = (sh.cols + V - 1) / V;
  const int rg = sh.threads / cg < p.d ? sh.threads / cg : p.d;
  const size_t smem = sizeof(float) * ((size_t)LS_SEG * ((GATE ? 3 : 2) * p.d + cg * V) + 2 * (size_t)rg * cg * V);
#define LS_GO(V_, NR_)                                                                                               \
  do {                                                                                                               \
    if (smem > 48 * 1024)                                                                                            \
      cudaFuncSetAttribute(ls_walk_kernel<T, GATE, V_, NR_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    rllm_launch_pdl(ls_walk_kernel<T, GATE, V_, NR_>, dim3(p.heads, num_seqs, gz), dim3(sh.threads), smem, stream, a, p, \
                    state, q_start, slots, num_slots, sh.cols, out, gz > 1 ? raw : (float*)nullptr, early, err);     \
  } while (0)
  if (V == 4) {
    if (sh.nr <= 4) LS_GO(4, 4);
    else if (sh.nr <= 8) LS_GO(4, 8);
    else LS_GO(4, 16);
  } else {
    if (sh.nr <= 8) LS_GO(1, 8);
    else LS_GO(1, 32);
  }
#undef LS_GO
  if (gz > 1) {
    const long long warps = (long long)T_tokens * p.heads;
    rllm_launch_pdl(ls_norm_kernel<T>, dim3((unsigned)((warps + 3) / 4)), dim3(128), (size_t)0, stream, (const float*)raw, a,
                    p, out, T_tokens);
  }
  return 0;
}

// a: T rows of [q: heads d | k or f: heads d | v: heads dv | (g: heads dv)] with row stride `stride`; out [T, heads dv].
// f_bias (and lower) given: decays per channel; else decay [heads].  early: the kernel launched directly ahead does
// not write `state`, so that it may be fetched while that one still runs.
RLLM_EXPORT int rllm_linear_state_walk(const void* a, int stride, int dtype, const float* decay, const double* inv_freq,
                                       int rd, float k_scale, const float* f_bias, const float* lower,
                                       const float* norm_w, float eps, int gated, const int* positions, float* state,
                                       const int* q_start, const int* slots, int num_slots, int num_seqs, int T,
                                       int heads, int d, int dv, void* out, float* raw, int early, int* err,
                                       cudaStream_t stream) {
  if (num_seqs <= 0 || T <= 0) return 0;
  if (heads <= 0 || d <= 0 || dv <= 0 || num_slots <= 0 || num_seqs > 65535) return RLLM_E_BADARG;
  if ((f_bias != nullptr) != (lower != nullptr) || (!f_bias && !decay)) return RLLM_E_BADARG;
  if (rd < 0 || rd > d || (rd & 1) || (rd > 0 && (!inv_freq || !positions))) return RLLM_E_BADARG;
  if (stride < heads * (2 * d + dv * (gated ? 2 : 1))) return RLLM_E_BADARG;
  const LsArgs p{stride, heads, d, dv, decay, inv_freq, rd, k_scale, f_bias, lower, norm_w, eps, gated, positions};
  int rc = 0;
  RLLM_DISPATCH_DTYPE(dtype, TT, {
    rc = f_bias ? ls_walk<TT, true>((const TT*)a, p, state, q_start, slots, num_slots, num_seqs, T, (TT*)out, raw, early, err, stream)
                : ls_walk<TT, false>((const TT*)a, p, state, q_start, slots, num_slots, num_seqs, T, (TT*)out, raw, early, err, stream);
  });
  if (rc) return rc;
  RLLM_LAUNCH_CHECK();
  return 0;
}

RLLM_EXPORT int rllm_linear_state_chunk() { return LSM_C; }
RLLM_EXPORT int rllm_linear_state_mma_takes(int d, int dv) { return d > 0 && dv > 0 && d <= 128 && dv <= 128 ? 1 : 0; }

// cosine and sine of every (token, pair) of a step: table [T, half] pairs of floats
RLLM_EXPORT int rllm_rotation_table(const int* positions, const double* inv_freq, int T, int half, void* table,
                                    cudaStream_t stream) {
  if (T <= 0 || half <= 0) return 0;
  const long long n = (long long)T * half;
  return (int)rllm_launch_pdl(ls_rotation_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), (size_t)0, stream,
                              positions, inv_freq, half, (float2*)table, n);
}

// The same over long portions of bfloat16 rows (linear_state_mma.cuh): chunks chunk0 .. chunk0 + max_chunks - 1 of every
// sequence's portion (a call goes on where the slots' states are), work num_seqs * max_chunks * heads * d * dv floats, gsum num_seqs * max_chunks * heads * d floats (decays per channel),
// table from rllm_rotation_table (fixed decays with rd > 0), indexed by the same tokens as a's rows.
RLLM_EXPORT int rllm_linear_state_chunked(const void* a, int stride, const float* decay, const void* table, int rd,
                                          float k_scale, const float* f_bias, const float* lower, const float* norm_w,
                                          float eps, int gated, float* state, float* work, float* gsum, const int* q_start,
                                          const int* slots, int num_slots, int num_seqs, int chunk0, int max_chunks, int heads,
                                          int d, int dv, void* out, int* err, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || d <= 0 || dv <= 0 || num_slots <= 0 || max_chunks <= 0 || chunk0 < 0 || !work || !state)
    return RLLM_E_BADARG;
  if ((f_bias != nullptr) != (lower != nullptr) || (!f_bias && !decay) || (f_bias && !gsum)) return RLLM_E_BADARG;
  if (rd < 0 || rd > d || (rd & 1) || (rd > 0 && !table) || stride < heads * (2 * d + dv * (gated ? 2 : 1))) return RLLM_E_BADARG;
  if (d > 128 || dv > 128 || (long long)num_seqs * max_chunks > 65535) return RLLM_E_UNSUPPORTED;
  const LsArgs p{stride, heads, d, dv, decay, nullptr, rd, k_scale, f_bias, lower, norm_w, eps, gated, nullptr};
#define LSM_GO(D_, DV_)                                                                                                      \
  (f_bias ? lsm_launch<D_, DV_, true>((const bf16*)a, p, (const float2*)table, state, work, gsum, q_start, slots, num_slots,  \
                                      num_seqs, chunk0, max_chunks, (bf16*)out, err, stream)                                         \
          : lsm_launch<D_, DV_, false>((const bf16*)a, p, (const float2*)table, state, work, gsum, q_start, slots, num_slots, \
                                       num_seqs, chunk0, max_chunks, (bf16*)out, err, stream))
  const int rc = d <= 64 ? (dv <= 64 ? LSM_GO(64, 64) : LSM_GO(64, 128)) : (dv <= 64 ? LSM_GO(128, 64) : LSM_GO(128, 128));
#undef LSM_GO
  if (rc) return rc;
  RLLM_LAUNCH_CHECK();
  return 0;
}
