// The gated delta rule with a decay per key channel.  Per head, with unit vectors q, k of size d (q already
// scaled), values v of size dv, decays g of size d and a step beta:
//
//   S' = diag(g_t) S_(t-1);   u_t = beta_t (v_t - S'^T k_t);   S_t = S' + k_t u_t^T   [d, dv];   o_t = S_t^T q_t
//
// S lives in float32 in the request's state slot [heads][d][dv], starts at zero and is carried from step to
// step.  Everything but the loads of the convolutions' results (which may be bfloat16) is float32 arithmetic.
//
//   channel_delta_prepare   per token: q and k of every q/k head over their Euclidean norms, the decays
//                           g = exp(-exp(a_log) softplus(step + dt_bias)) and beta = sigmoid(b), as float32
//                           arrays that the scan then only copies.
//   channel_delta_walk      a block owns 16 value columns of a head of a sequence: the columns of S never meet,
//                           so eight lanes keep one column (every eighth group of four rows each) in
//                           registers and walk the tokens of the step in order; the two sums over the rows
//                           are shuffles among the eight.  Tokens come through shared memory in segments of 16
//                           that are copied ahead (cp.async, two buffers).  A token's result does not depend
//                           on how the sequence was cut or on the batch.
//   channel_delta_step      one token of every sequence (decoding): a block a (head, sequence) does everything
//                           between the mixer's first product and its last: the convolutions (where no two heads
//                           share a q/k head), unit vectors, the decays' and the gate's low-rank second products,
//                           beta's product, the recurrence, the head's norm and its gate.
//   channel_delta_records / _chunks   long portions of bfloat16 activations, sixteen tokens at a time on the tensor
//                           cores: see channel_delta_mma.cuh.
#include "common.cuh"
#include "channel_delta_mma.cuh"
#include <math.h>

#define CD_MAX_D 256
#define CD_COLS 16              // value columns a block owns
#define CD_LANES 8              // lanes that share a column
#define CD_SEG 16               // tokens a segment

__device__ __forceinline__ float cd_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float cd_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

// One warp an item of a token: items 0 .. kv - 1 are the q heads, .. 2 kv - 1 the k heads, then the heads' decays.
// c: rows [q: kv d | k: kv d | ...]; step [T, heads d]; b [T, heads]; qn, kn [T, kv, d]; g [T, heads, d].
template <typename T>
__global__ void __launch_bounds__(128)
channel_delta_prepare_kernel(const T* c, int c_stride, const float* step, const float* b, const float* dt_bias,
                             const float* a_log, float* qn, float* kn, float* g, float* beta, int T_tokens, int heads,
                             int kv, int d, float unit_eps, float qscale) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31;
  const int items = 2 * kv + heads;
  const long long gw = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (gw >= (long long)T_tokens * items) return;
  const int t = (int)(gw / items), it = (int)(gw - (long long)t * items);
  if (it < 2 * kv) {
    const T* src = c + (size_t)t * c_stride + (size_t)it * d;
    float* dst = (it < kv ? qn + ((size_t)t * kv + it) * d : kn + ((size_t)t * kv + it - kv) * d);
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) { const float v = to_f32(src[i]); ss = fmaf(v, v, ss); }
    ss = warp_sum(ss);
    const float r = (it < kv ? qscale : 1.0f) / sqrtf(ss + unit_eps);
    for (int i = lane; i < d; i += 32) dst[i] = to_f32(src[i]) * r;
    return;
  }
  const int h = it - 2 * kv;
  const float rate = expf(a_log[h]);
  const float* st = step + ((size_t)t * heads + h) * d;
  float* gd = g + ((size_t)t * heads + h) * d;
  for (int i = lane; i < d; i += 32) gd[i] = expf(-rate * cd_softplus(st[i] + dt_bias[h * d + i]));
  if (lane == 0) beta[(size_t)t * heads + h] = cd_sigmoid(b[(size_t)t * heads + h]);
}

__device__ __forceinline__ void cd_copy16(float* dst, const float* src) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ void cd_copy4(float* dst, const float* src) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(a), "l"(src) : "memory");
}
__device__ __forceinline__ void cd_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cd_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// R: rows of S a thread keeps (d <= 8 R)
template <typename T, int R>
__global__ void __launch_bounds__(CD_COLS * CD_LANES)
channel_delta_walk_kernel(const float* qn, const float* kn, const float* g, const float* beta, const T* v,
                          int v_stride, float* state, const int* q_start, const int* slots, int num_slots, float* out,
                          int heads, int per, int d, int dv, int* err) {
  constexpr int DP = CD_LANES * R;                       // rows with the padding
  extern __shared__ __align__(16) float sm[];
  float* buf = sm;                                       // [2][3: k, q, g][CD_SEG][DP]
  float* vs = sm + 2 * 3 * CD_SEG * DP;                  // [2][CD_SEG][CD_COLS]
  float* bs = vs + 2 * CD_SEG * CD_COLS;                 // [2][CD_SEG]
  float* os = bs + 2 * CD_SEG;                           // [CD_SEG][CD_COLS]
  pdl_wait();
  pdl_launch();
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * CD_COLS;
  const int t0 = q_start[s], t1 = q_start[s + 1];
  if (t1 <= t0) return;
  const int slot = slots[s];
  if (slot < 0 || slot >= num_slots) {
    if (threadIdx.x == 0) atomicOr(err, 8);
    return;
  }
  const int tid = threadIdx.x, l = tid & (CD_LANES - 1), cl = tid / CD_LANES, col = col0 + cl;
  const bool live = col < dv;
  const int kvh = h / per, kv = heads / per;
  float* sp = state + ((size_t)slot * heads + h) * d * dv;
  for (int i = tid; i < 2 * 3 * CD_SEG * DP; i += blockDim.x) buf[i] = 0.f;     // the padding rows stay zero
  float S[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = 4 * (l + CD_LANES * (i >> 2)) + (i & 3);
    S[i] = (live && r < d) ? sp[(size_t)r * dv + col] : 0.f;
  }
  __syncthreads();
  const bool wide = (d & 3) == 0;
  T pv[CD_SEG * CD_COLS / (CD_COLS * CD_LANES)];
  float pb = 0.f;
  auto fetch = [&](int seg, int which) {                 // a segment's rows on their way into buffer `which`
    const int n = min(CD_SEG, t1 - seg);
    float* kb = buf + (size_t)which * 3 * CD_SEG * DP;
    if (wide) {
      const int q4 = d >> 2;
      for (int e = tid; e < n * q4; e += blockDim.x) {
        const int x = e / q4, i = (e - x * q4) * 4;
        const size_t at = ((size_t)(seg + x) * kv + kvh) * d + i;
        cd_copy16(kb + x * DP + i, kn + at);
        cd_copy16(kb + (CD_SEG + x) * DP + i, qn + at);
        cd_copy16(kb + (2 * CD_SEG + x) * DP + i, g + ((size_t)(seg + x) * heads + h) * d + i);
      }
    } else {
      for (int e = tid; e < n * d; e += blockDim.x) {
        const int x = e / d, i = e - x * d;
        const size_t at = ((size_t)(seg + x) * kv + kvh) * d + i;
        cd_copy4(kb + x * DP + i, kn + at);
        cd_copy4(kb + (CD_SEG + x) * DP + i, qn + at);
        cd_copy4(kb + (2 * CD_SEG + x) * DP + i, g + ((size_t)(seg + x) * heads + h) * d + i);
      }
    }
    cd_commit();
#pragma unroll
    for (int u = 0; u < (int)(sizeof(pv) / sizeof(T)); ++u) {
      const int e = tid + u * CD_COLS * CD_LANES, x = e / CD_COLS, c = e - x * CD_COLS;
      pv[u] = (x < n && col0 + c < dv) ? v[(size_t)(seg + x) * v_stride + (size_t)h * dv + col0 + c] : from_f32<T>(0.f);
    }
    if (tid < n) pb = beta[(size_t)(seg + tid) * heads + h];
  };
  auto land = [&](int which) {                           // the fetched values and steps into shared memory
#pragma unroll
    for (int u = 0; u < (int)(sizeof(pv) / sizeof(T)); ++u) vs[which * CD_SEG * CD_COLS + tid + u * CD_COLS * CD_LANES] = to_f32(pv[u]);
    if (tid < CD_SEG) bs[which * CD_SEG + tid] = pb;
  };
  fetch(t0, 0);
  land(0);
  int which = 0;
  for (int seg = t0; seg < t1; seg += CD_SEG, which ^= 1) {
    const int n = min(CD_SEG, t1 - seg);
    const bool more = seg + CD_SEG < t1;
    if (more) { fetch(seg + CD_SEG, which ^ 1); cd_wait<1>(); } else { cd_wait<0>(); }
    __syncthreads();
    const float* kb = buf + (size_t)which * 3 * CD_SEG * DP + 4 * l;
#pragma unroll 1
    for (int x = 0; x < n; ++x) {
      const float* kr = kb + x * DP;
      float a0 = 0.f, a1 = 0.f, a2 = 0.f, a3 = 0.f;
      float4 kk[R / 4];
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        kk[i] = *(const float4*)(kr + 4 * CD_LANES * i);
        const float4 gg = *(const float4*)(kr + 2 * CD_SEG * DP + 4 * CD_LANES * i);
        S[4 * i + 0] *= gg.x; S[4 * i + 1] *= gg.y; S[4 * i + 2] *= gg.z; S[4 * i + 3] *= gg.w;
        a0 = fmaf(S[4 * i + 0], kk[i].x, a0); a1 = fmaf(S[4 * i + 1], kk[i].y, a1);
        a2 = fmaf(S[4 * i + 2], kk[i].z, a2); a3 = fmaf(S[4 * i + 3], kk[i].w, a3);
      }
      float dot = (a0 + a1) + (a2 + a3);
#pragma unroll
      for (int o = CD_LANES / 2; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
      const float u = bs[which * CD_SEG + x] * (vs[(which * CD_SEG + x) * CD_COLS + cl] - dot);
      a0 = a1 = a2 = a3 = 0.f;
#pragma unroll
      for (int i = 0; i < R / 4; ++i) {
        const float4 qq = *(const float4*)(kr + CD_SEG * DP + 4 * CD_LANES * i);
        S[4 * i + 0] = fmaf(kk[i].x, u, S[4 * i + 0]); S[4 * i + 1] = fmaf(kk[i].y, u, S[4 * i + 1]);
        S[4 * i + 2] = fmaf(kk[i].z, u, S[4 * i + 2]); S[4 * i + 3] = fmaf(kk[i].w, u, S[4 * i + 3]);
        a0 = fmaf(S[4 * i + 0], qq.x, a0); a1 = fmaf(S[4 * i + 1], qq.y, a1);
        a2 = fmaf(S[4 * i + 2], qq.z, a2); a3 = fmaf(S[4 * i + 3], qq.w, a3);
      }
      float o = (a0 + a1) + (a2 + a3);
#pragma unroll
      for (int w = CD_LANES / 2; w > 0; w >>= 1) o += __shfl_xor_sync(0xffffffffu, o, w);
      if (l == 0) os[x * CD_COLS + cl] = o;
    }
    if (more) land(which ^ 1);
    __syncthreads();                                     // everybody is through with this buffer; outputs are in
    for (int e = tid; e < n * CD_COLS; e += blockDim.x) {
      const int x = e / CD_COLS, c = e - x * CD_COLS;
      if (col0 + c < dv) out[((size_t)(seg + x) * heads + h) * dv + col0 + c] = os[e];
    }
    // (the next segment's first outputs go into os only behind the next barrier)
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = 4 * (l + CD_LANES * (i >> 2)) + (i & 3);
    if (live && r < d) sp[(size_t)r * dv + col] = S[i];
  }
}

// The second product of a low-rank pair, one row: w [rank] . x [rank] (rank a multiple of 8, rows 16-byte aligned)
template <typename T>
__device__ __forceinline__ float cd_low_rank(const T* w, const float* xs, int rank) {
  constexpr int V = 16 / sizeof(T);
  float acc[2] = {0.f, 0.f};
#pragma unroll 4
  for (int i = 0; i < rank; i += V) {
    struct alignas(16) A { T v[V]; };
    const A a = *(const A*)(w + i);
#pragma unroll
    for (int y = 0; y < V; ++y) acc[y & 1] = fmaf(to_f32(a.v[y]), xs[i + y], acc[y & 1]);
  }
  return acc[0] + acc[1];
}

struct CdStep {
  const void* a;             // [S, .]: the first product: q | k | v, W_a1 h at at_a, W_g1 h at at_g
  const void* c;             // [S, channels]: the convolutions' results (null: made here)
  const void* x;             // [S, H]: the mixer's input
  const void *w_b, *w_a2, *w_g2, *w_conv;
  const float *dt_bias, *a_log, *norm;
  float *tail, *state;       // [slots, taps - 1, channels]; [slots, heads, d, dv]
  const int* slots;
  void* out;                 // [S, heads dv]
  int a_stride, x_stride, at_a, at_g, rank_a, rank_g, H, taps, num_slots, heads, kv, d, dv;
  float unit_eps, qscale, eps;
  int early;
};

// RW: rows of S a warp keeps (d <= 8 RW); NC: groups of 128 value columns.  TC: the convolution weights' type.
template <typename T, typename TC, int RW, int NC>
__global__ void __launch_bounds__(256)
channel_delta_step_kernel(CdStep p, int* err) {
  __shared__ float qs[8 * RW], ks[8 * RW], gs[8 * RW], vs[128 * NC], gate_s[128 * NC];
  __shared__ __align__(16) float us[128 * NC];
  __shared__ __align__(16) float red[8][128 * NC];
  __shared__ float red32[32], beta_s;
  extern __shared__ float low[];                         // the two low-rank inputs
  const int h = blockIdx.x, s = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int d = p.d, dv = p.dv, kvh = h / (p.heads / p.kv), channels = 2 * p.kv * d + p.heads * dv;
  const int slot = p.slots[s];
  if (slot < 0 || slot >= p.num_slots) {
    pdl_wait();
    pdl_launch();
    if (tid == 0) atomicOr(err, 8);
    return;
  }
  // `early`: the kernel directly ahead does not write the state, so its loads need not wait for that kernel
  if (!p.early) pdl_wait();
  float* sp = p.state + ((size_t)slot * p.heads + h) * d * dv;
  float4 S[RW][NC];
#pragma unroll
  for (int i = 0; i < RW; ++i)
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int row = warp * RW + i, col = 4 * lane + 128 * c;
      S[i][c] = (row < d && col < dv) ? *(const float4*)(sp + (size_t)row * dv + col) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  pdl_wait();
  pdl_launch();
  const T* ar = (const T*)p.a + (size_t)s * p.a_stride;
  // q, k, v of this head after their convolutions
  for (int e = tid; e < 2 * d + dv; e += 256) {
    const int ch = e < d ? kvh * d + e : (e < 2 * d ? (p.kv + kvh) * d + e - d : 2 * p.kv * d + h * dv + e - 2 * d);
    float val;
    if (p.c) {
      val = to_f32(((const T*)p.c)[(size_t)s * channels + ch]);
    } else {
      const TC* w = (const TC*)p.w_conv + (size_t)ch * p.taps;
      float* tl = p.tail + (size_t)slot * (p.taps - 1) * channels + ch;
      const float now = to_f32(ar[ch]);
      float acc = to_f32(w[p.taps - 1]) * now;
      for (int j = 0; j + 1 < p.taps; ++j) {             // the inputs ahead, moved on by one on the way
        const float v = tl[(size_t)j * channels];
        acc = fmaf(to_f32(w[j]), v, acc);
        if (j > 0) tl[(size_t)(j - 1) * channels] = v;
      }
      if (p.taps > 1) tl[(size_t)(p.taps - 2) * channels] = now;
      val = to_f32(from_f32<T>(acc * cd_sigmoid(acc)));  // an activation, as the convolution kernel leaves it
    }
    if (e < d) qs[e] = val; else if (e < 2 * d) ks[e - d] = val; else vs[e - 2 * d] = val;
  }
  for (int e = tid; e < p.rank_a + p.rank_g; e += 256) low[e] = to_f32(ar[e < p.rank_a ? p.at_a + e : p.at_g + e - p.rank_a]);
  float bd = 0.f;
  const T* xr = (const T*)p.x + (size_t)s * p.x_stride;
  const T* wb = (const T*)p.w_b + (size_t)h * p.H;
  for (int i = tid; i < p.H; i += 256) bd = fmaf(to_f32(xr[i]), to_f32(wb[i]), bd);
  bd = block_sum(bd, red32);                             // (behind its barriers q, k, v and the low-rank inputs are in)
  if (tid == 0) beta_s = cd_sigmoid(bd);
  const float rate = expf(p.a_log[h]);
  for (int e = tid; e < d + dv; e += 256) {
    if (e < d) {
      const float z = cd_low_rank((const T*)p.w_a2 + ((size_t)h * d + e) * p.rank_a, low, p.rank_a) + p.dt_bias[h * d + e];
      gs[e] = expf(-rate * cd_softplus(z));
    } else {
      const float z = cd_low_rank((const T*)p.w_g2 + ((size_t)h * dv + e - d) * p.rank_g, low + p.rank_a, p.rank_g);
      gate_s[e - d] = cd_sigmoid(to_f32(from_f32<T>(z)));
    }
  }
  float q2 = 0.f, k2 = 0.f;
  for (int i = lane; i < d; i += 32) { q2 = fmaf(qs[i], qs[i], q2); k2 = fmaf(ks[i], ks[i], k2); }
  const float rq = p.qscale / sqrtf(warp_sum(q2) + p.unit_eps), rk = 1.0f / sqrtf(warp_sum(k2) + p.unit_eps);
  __syncthreads();
  float4 acc[NC];
#pragma unroll
  for (int c = 0; c < NC; ++c) acc[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < RW; ++i) {
    const int row = warp * RW + i;
    const float g = row < d ? gs[row] : 0.f, k = row < d ? ks[row] * rk : 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      S[i][c].x *= g; S[i][c].y *= g; S[i][c].z *= g; S[i][c].w *= g;
      acc[c].x = fmaf(S[i][c].x, k, acc[c].x); acc[c].y = fmaf(S[i][c].y, k, acc[c].y);
      acc[c].z = fmaf(S[i][c].z, k, acc[c].z); acc[c].w = fmaf(S[i][c].w, k, acc[c].w);
    }
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) *(float4*)&red[warp][4 * lane + 128 * c] = acc[c];
  __syncthreads();
  for (int j = tid; j < dv; j += 256) {
    float dot = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) dot += red[w][j];
    us[j] = beta_s * (vs[j] - dot);
  }
  __syncthreads();
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = 4 * lane + 128 * c;
    const float4 u = col < dv ? *(const float4*)&us[col] : make_float4(0.f, 0.f, 0.f, 0.f);
    acc[c] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < RW; ++i) {
      const int row = warp * RW + i;
      const float k = row < d ? ks[row] * rk : 0.f, q = row < d ? qs[row] * rq : 0.f;
      S[i][c].x = fmaf(k, u.x, S[i][c].x); S[i][c].y = fmaf(k, u.y, S[i][c].y);
      S[i][c].z = fmaf(k, u.z, S[i][c].z); S[i][c].w = fmaf(k, u.w, S[i][c].w);
      acc[c].x = fmaf(S[i][c].x, q, acc[c].x); acc[c].y = fmaf(S[i][c].y, q, acc[c].y);
      acc[c].z = fmaf(S[i][c].z, q, acc[c].z); acc[c].w = fmaf(S[i][c].w, q, acc[c].w);
      if (row < d && col < dv) *(float4*)(sp + (size_t)row * dv + col) = S[i][c];
    }
    *(float4*)&red[warp][col] = acc[c];
  }
  __syncthreads();
  float o = 0.f;
  if (tid < dv) {
#pragma unroll
    for (int w = 0; w < 8; ++w) o += red[w][tid];
  }
  const float ss = block_sum(o * o, red32);
  if (tid < dv)
    ((T*)p.out)[((size_t)s * p.heads + h) * dv + tid] =
        from_f32<T>(o / sqrtf(ss / (float)dv + p.eps) * p.norm[tid] * gate_s[tid]);
}

// Whether the one-token kernel takes these sizes
RLLM_EXPORT int rllm_channel_delta_step_takes(int d, int dv, int rank_a, int rank_g) {
  return d <= 128 && dv <= 256 && dv % 4 == 0 && rank_a % 8 == 0 && rank_g % 8 == 0 && rank_a + rank_g <= 2048;
}

RLLM_EXPORT int rllm_channel_delta_step(const void* a, int a_stride, const void* c, const void* x, int x_stride,
                                        const void* w_b, const void* w_a2, const void* w_g2, const void* w_conv,
                                        int conv_dtype, const float* dt_bias, const float* a_log, const float* norm,
                                        float* tail, float* state, const int* slots, void* out, int dtype, int num_seqs,
                                        int at_a, int at_g, int rank_a, int rank_g, int H, int taps, int num_slots,
                                        int heads, int kv, int d, int dv, float unit_eps, float qscale, float eps, int early,
                                        int* err, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || kv <= 0 || heads % kv || d <= 0 || dv <= 0 || num_slots <= 0 || taps < 1) return RLLM_E_BADARG;
  if (!c && kv != heads) return RLLM_E_BADARG;            // a q/k head that two blocks share: they would both move its inputs on
  if (!rllm_channel_delta_step_takes(d, dv, rank_a, rank_g) || heads > 65535 || num_seqs > 65535) return RLLM_E_UNSUPPORTED;
  CdStep p{a, c, x, w_b, w_a2, w_g2, w_conv, dt_bias, a_log, norm, tail, state, slots, out, a_stride, x_stride, at_a, at_g,
           rank_a, rank_g, H, taps, num_slots, heads, kv, d, dv, unit_eps, qscale, eps, early};
#define CDS_GO(T_, TC_, RW_, NC_)                                                                                       \
  rllm_launch_pdl(channel_delta_step_kernel<T_, TC_, RW_, NC_>, dim3(heads, num_seqs), dim3(256),                        \
                  (size_t)(rank_a + rank_g) * sizeof(float), stream, p, err)
  RLLM_DISPATCH_DTYPE(dtype, TT, RLLM_DISPATCH_DTYPE(conv_dtype, TC, {
    if (d <= 64) { if (dv <= 128) CDS_GO(TT, TC, 8, 1); else CDS_GO(TT, TC, 8, 2); }
    else { if (dv <= 128) CDS_GO(TT, TC, 16, 1); else CDS_GO(TT, TC, 16, 2); }
  }));
#undef CDS_GO
  RLLM_LAUNCH_CHECK();
  return 0;
}

RLLM_EXPORT int rllm_channel_delta_prepare(const void* c, int c_stride, int dtype, const float* step, const float* b,
                                           const float* dt_bias, const float* a_log, float* qn, float* kn, float* g,
                                           float* beta, int T, int heads, int kv, int d, float unit_eps, float qscale,
                                           cudaStream_t stream) {
  if (T <= 0) return 0;
  if (heads <= 0 || kv <= 0 || heads % kv || d <= 0) return RLLM_E_BADARG;
  const long long warps = (long long)T * (2 * kv + heads);
  RLLM_DISPATCH_DTYPE(dtype, TT,
    (rllm_launch_pdl(channel_delta_prepare_kernel<TT>, dim3((unsigned)((warps + 3) / 4)), dim3(128), (size_t)0, stream,
                     (const TT*)c, c_stride, step, b, dt_bias, a_log, qn, kn, g, beta, T, heads, kv, d, unit_eps, qscale)));
  RLLM_LAUNCH_CHECK();
  return 0;
}

RLLM_EXPORT int rllm_channel_delta_walk(const float* qn, const float* kn, const float* g, const float* beta,
                                        const void* v, int v_stride, int dtype, float* state, const int* q_start,
                                        const int* slots, int num_slots, int num_seqs, float* out, int heads, int kv,
                                        int d, int dv, int* err, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || kv <= 0 || heads % kv || d <= 0 || dv <= 0 || num_slots <= 0) return RLLM_E_BADARG;
  if (d > CD_MAX_D || heads > 65535 || num_seqs > 65535) return RLLM_E_UNSUPPORTED;
#define CD_GO(T_, R_)                                                                                              \
  do {                                                                                                             \
    const size_t smem = (2 * 3 * CD_SEG * CD_LANES * (R_) + 3 * CD_SEG * CD_COLS + 2 * CD_SEG) * sizeof(float);     \
    if (smem > 48 * 1024)                                                                                          \
      cudaFuncSetAttribute(channel_delta_walk_kernel<T_, R_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    rllm_launch_pdl(channel_delta_walk_kernel<T_, R_>, dim3((dv + CD_COLS - 1) / CD_COLS, heads, num_seqs),         \
                    dim3(CD_COLS * CD_LANES), smem, stream, qn, kn, g, beta, (const T_*)v, v_stride, state, q_start, \
                    slots, num_slots, out, heads, heads / kv, d, dv, err);                                         \
  } while (0)
  RLLM_DISPATCH_DTYPE(dtype, TT, {
    if (d <= 32) CD_GO(TT, 4);
    else if (d <= 64) CD_GO(TT, 8);
    else if (d <= 128) CD_GO(TT, 16);
    else CD_GO(TT, 32);
  });
#undef CD_GO
  RLLM_LAUNCH_CHECK();
  return 0;
}

// Bytes of workspace a (chunk of 16 tokens, head) takes in the chunked form; 0: no such form for this head.
static inline int cdm_size(int d) { return d <= 64 ? 64 : (d <= 128 ? 128 : 0); }
RLLM_EXPORT int rllm_channel_delta_chunk_bytes(int d, int dv) {
  const int D = cdm_size(d);
  if (!D || d <= 0 || dv <= 0) return 0;
  const int rec = D == 64 ? (int)sizeof(CdmRecord<64>) : (int)sizeof(CdmRecord<128>);
  return rec + (dv + 15) / 16 * 16 * CDM_CHUNK * (int)sizeof(float);
}

// Chunks chunk0 .. chunk0 + seg - 1 of every sequence (a chunk: 16 tokens of the step, counted from the sequence's
// first): two launches.  Calls for rising chunk0 carry the state from one to the next through the slots.
// work: num_seqs * seg * heads * rllm_channel_delta_chunk_bytes.
RLLM_EXPORT int rllm_channel_delta_chunked(const void* c, int c_stride, const float* step, const float* b,
                                           const float* dt_bias, const float* a_log, float unit_eps, float qscale,
                                           float* state, const int* q_start, const int* slots, int num_slots,
                                           int num_seqs, int chunk0, int seg, void* work, float* out, int heads, int kv,
                                           int d, int dv, int* err, cudaStream_t stream) {
  if (num_seqs <= 0 || seg <= 0) return 0;
  if (heads <= 0 || kv <= 0 || heads % kv || d <= 0 || dv <= 0 || num_slots <= 0 || chunk0 < 0 || !work) return RLLM_E_BADARG;
  if (!cdm_size(d) || heads > 65535 || (long long)num_seqs * seg > 65535 || num_seqs > 65535) return RLLM_E_UNSUPPORTED;
  const int dvp = (dv + 15) / 16 * 16;
#define CDM_GO(D_)                                                                                                   \
  do {                                                                                                               \
    CdmRecord<D_>* rec = (CdmRecord<D_>*)work;                                                                       \
    float* u0 = (float*)(rec + (size_t)num_seqs * seg * heads);                                                      \
    rllm_launch_pdl(channel_delta_records_kernel<D_>, dim3(heads, num_seqs * seg), dim3(CDM_PREP_THREADS), (size_t)0, \
                    stream, (const bf16*)c, c_stride, step, b, dt_bias, a_log, q_start, chunk0, seg, rec, u0, heads, \
                    kv, d, dv, dvp, unit_eps, qscale);                                                               \
    const size_t smem = sizeof(CdmSmem<D_>);                                                                         \
    static bool allowed = false;                                                                                     \
    if (!allowed) {                                                                                                  \
      cudaFuncSetAttribute(channel_delta_chunks_kernel<D_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
      allowed = true;                                                                                                \
    }                                                                                                                \
    /* an ordinary launch: blocks that came in early, as records' blocks leave, would share SMs while others idle */  \
    channel_delta_chunks_kernel<D_><<<dim3(dvp / 16, heads, num_seqs), dim3(CDM_THREADS), smem, stream>>>(           \
        rec, u0, state, q_start, slots, num_slots, chunk0, seg, out, heads, d, dv, dvp, err);                        \
  } while (0)
  if (cdm_size(d) == 64) CDM_GO(64); else CDM_GO(128);
#undef CDM_GO
  RLLM_LAUNCH_CHECK();
  return 0;
}
