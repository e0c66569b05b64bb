// What stands between the sublayers of a layer whose sublayer results are gated
// and normalised before they join the residual stream, and whose stream is a
// weighted sum of the results of all layers so far.  All arithmetic is float32;
// the stream and the layer results are float32 in memory.
//
//   gated_postnorm_add:  v = (sum_k c[t, k] y[t, k, :]) * sigmoid(g[t, :] + b)      (g absent: no gate)
//                        x_out[t, :] = x_in[t, :] + v / sqrt(mean(v^2) + eps) * w
//                        and, if asked, next[t, :] = x_out / sqrt(mean(x_out^2) + eps2) * w2
//                        (the norm that reads the stream next).  With a history of layer results
//                        (x_out being its last level) the depth average follows in the same kernel:
//                        s = sum_j a[j] X[j, t, :] is written as the stream and the next norm reads s.
//   depth_average:       s[r, :] = sum_j a[j] X[j, row(r), :], the stream itself and/or
//                        its RMS norm in the activation dtype; row(r) = rows[r] or r.
//   postnorm_add:        v = s0 y0[t, :] (+ s1 y1[t, :]);  x[t, :] += c v / sqrt(mean(v^2) + eps) * w, in place,
//                        and the new x in the activation dtype beside it (what the next sublayer reads)
//   activation_rows:     the stream in the activation dtype;   scaled_sum2: s0 a + s1 b
// One block per row; the order of a row's additions depends on H and the block
// size only.
#include "common.cuh"

#define GLUE_THREADS 256

template <typename TA, typename TW>
__global__ void __launch_bounds__(GLUE_THREADS)
gated_postnorm_add_kernel(const float* x_in, float* x_out, const TA* y,
                          int slots, const float* slot_w, const TA* g, int g_stride,
                          const TW* gb, const TW* nw, float eps,
                          const TW* next_w, TA* next_out, float next_eps, const float* hist,
                          long long level_stride, int levels, const TW* coeff, float* stream_out, int H) {
  // (Every kernel of this file starts with the wait for the kernel ahead of it in the stream and lets the
  // next one in right after: launches overlap the tails of their predecessors.  The pointer parameters
  // carry no __restrict__, so that no load is proved independent of that wait and moved above it.)
  pdl_wait();
  pdl_launch();
  extern __shared__ float row[];
  __shared__ float red[32];
  const int t = blockIdx.x;
  const TA* gr = g + (size_t)t * g_stride;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v;
    if (slot_w == nullptr) {
      v = to_f32(y[(size_t)t * H + i]);
    } else {
      v = 0.f;
      for (int k = 0; k < slots; ++k)
        v = fmaf(slot_w[(size_t)t * slots + k], to_f32(y[((size_t)t * slots + k) * H + i]), v);
    }
    if (g != nullptr) {                                  // no gate: the sublayer's result as it is
      const float a = to_f32(gr[i]) + (gb ? to_f32(gb[i]) : 0.f);
      v *= 1.0f / (1.0f + expf(-a));
    }
    row[i] = v;
    ss += v * v;
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  float ss2 = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float xn = x_in[(size_t)t * H + i] + row[i] * inv * to_f32(nw[i]);
    x_out[(size_t)t * H + i] = xn;
    if (hist != nullptr) {
      // the depth average in the order of depth_average_kernel; x_out is the history's last level
      float s = 0.f;
      for (int j = 0; j + 1 < levels; ++j) s = fmaf(to_f32(coeff[j]), hist[(size_t)j * level_stride + (size_t)t * H + i], s);
      xn = fmaf(to_f32(coeff[levels - 1]), xn, s);
      stream_out[(size_t)t * H + i] = xn;
    }
    row[i] = xn;
    ss2 += xn * xn;
  }
  if (next_w == nullptr) return;
  ss2 = block_sum(ss2, red);
  const float inv2 = 1.0f / sqrtf(ss2 / (float)H + next_eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    next_out[(size_t)t * H + i] = from_f32<TA>(row[i] * inv2 * to_f32(next_w[i]));
}

RLLM_EXPORT int rllm_gated_postnorm_add(const float* x_in, float* x_out, const void* y, int slots,
                                        const float* slot_w, const void* g, int g_stride, const void* gb,
                                        const void* nw, float eps, const void* next_w, void* next_out,
                                        float next_eps, const float* hist, long long level_stride, int levels,
                                        const void* coeff, float* stream_out, int T, int H, int act_dtype,
                                        int w_dtype, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || slots < 1 || (g != nullptr && g_stride < H)) return RLLM_E_BADARG;
  if (hist != nullptr && (levels < 1 || coeff == nullptr || stream_out == nullptr)) return RLLM_E_BADARG;
  const size_t smem = (size_t)H * sizeof(float);
  if (smem > 200 * 1024) return RLLM_E_UNSUPPORTED;
#define GLUE_LAUNCH(TA, TW)                                                                              \
  do {                                                                                                   \
    if (smem > 48 * 1024)                                                                                \
      cudaFuncSetAttribute(gated_postnorm_add_kernel<TA, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                           (int)smem);                                                                   \
    rllm_launch_pdl(gated_postnorm_add_kernel<TA, TW>, dim3(T), dim3(GLUE_THREADS), (size_t)(smem), stream,                                 \
        x_in, x_out, (const TA*)y, slots, slot_w, (const TA*)g, g_stride, (const TW*)gb, (const TW*)nw,  \
        eps, (const TW*)next_w, (TA*)next_out, next_eps, hist, level_stride, levels, (const TW*)coeff, stream_out, H);                                             \
  } while (0)
  RLLM_DISPATCH_DTYPE(act_dtype, TA_, RLLM_DISPATCH_DTYPE(w_dtype, TW_, GLUE_LAUNCH(TA_, TW_)));
#undef GLUE_LAUNCH
  RLLM_LAUNCH_CHECK();
  return 0;
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(GLUE_THREADS)
depth_average_kernel(const float* hist, long long level_stride, int levels,
                     const TW* a, const int* rows, float* stream_out,
                     const TW* nw, TA* norm_out, float eps, int H) {
  pdl_wait();
  pdl_launch();
  extern __shared__ float row[];
  __shared__ float red[32];
  const int r = blockIdx.x;
  const int src = rows ? rows[r] : r;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float s = 0.f;
    for (int j = 0; j < levels; ++j) s = fmaf(to_f32(a[j]), hist[(size_t)j * level_stride + (size_t)src * H + i], s);
    if (stream_out) stream_out[(size_t)r * H + i] = s;
    row[i] = s;
    ss += s * s;
  }
  if (nw == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x)
    norm_out[(size_t)r * H + i] = from_f32<TA>(row[i] * inv * to_f32(nw[i]));
}

RLLM_EXPORT int rllm_depth_average(const float* hist, long long level_stride, int levels, const void* a,
                                   const int* rows, float* stream_out, const void* nw, void* norm_out,
                                   float eps, int R, int H, int act_dtype, int w_dtype, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (H <= 0 || levels < 1) return RLLM_E_BADARG;
  const size_t smem = (size_t)H * sizeof(float);
  if (smem > 200 * 1024) return RLLM_E_UNSUPPORTED;
#define GLUE_LAUNCH(TA, TW)                                                                            \
  do {                                                                                                 \
    if (smem > 48 * 1024)                                                                              \
      cudaFuncSetAttribute(depth_average_kernel<TA, TW>, cudaFuncAttributeMaxDynamicSharedMemorySize,  \
                           (int)smem);                                                                 \
    rllm_launch_pdl(depth_average_kernel<TA, TW>, dim3(R), dim3(GLUE_THREADS), (size_t)(smem), stream,                                    \
        hist, level_stride, levels, (const TW*)a, rows, stream_out, (const TW*)nw, (TA*)norm_out, eps, H); \
  } while (0)
  RLLM_DISPATCH_DTYPE(act_dtype, TA_, RLLM_DISPATCH_DTYPE(w_dtype, TW_, GLUE_LAUNCH(TA_, TW_)));
#undef GLUE_LAUNCH
  RLLM_LAUNCH_CHECK();
  return 0;
}

// A thread keeps its values of the row between the two passes: PN_KEEP groups of V neighbouring elements (the
// rest of very wide rows is read again).
#define PN_KEEP 4
template <typename T, int V> __device__ __forceinline__ void pn_load(const T* p, float (&o)[V]) {
  if (V == 1) { o[0] = to_f32(p[0]); return; }
  struct alignas(V * sizeof(T)) A { T v[V]; };
  const A a = *(const A*)p;
#pragma unroll
  for (int i = 0; i < V; ++i) o[i] = to_f32(a.v[i]);
}
template <typename T, int V> __device__ __forceinline__ void pn_store(T* p, const float (&o)[V]) {
  if (V == 1) { p[0] = from_f32<T>(o[0]); return; }
  struct alignas(V * sizeof(T)) A { T v[V]; };
  A a;
#pragma unroll
  for (int i = 0; i < V; ++i) a.v[i] = from_f32<T>(o[i]);
  *(A*)p = a;
}

template <typename TA, typename TW, int V>
__global__ void __launch_bounds__(GLUE_THREADS)
postnorm_add_kernel(float* x, const TA* y0, const TA* y1, float s0, float s1, const TW* w, float eps, float mult,
                    TA* x_act, int H) {
  pdl_wait();
  pdl_launch();
  __shared__ float red[32];
  const size_t base = (size_t)blockIdx.x * H;
  const int groups = H / V;
  float keep[PN_KEEP][V];
  auto value = [&](int g, float (&o)[V]) {
    pn_load<TA, V>(y0 + base + (size_t)g * V, o);
#pragma unroll
    for (int i = 0; i < V; ++i) o[i] *= s0;
    if (y1) {
      float b[V];
      pn_load<TA, V>(y1 + base + (size_t)g * V, b);
#pragma unroll
      for (int i = 0; i < V; ++i) o[i] = fmaf(s1, b[i], o[i]);
    }
  };
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < PN_KEEP; ++u) {
    const int g = threadIdx.x + u * blockDim.x;
    if (g < groups) {
      value(g, keep[u]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss = fmaf(keep[u][i], keep[u][i], ss);
    }
  }
  for (int g = threadIdx.x + PN_KEEP * blockDim.x; g < groups; g += blockDim.x) {
    float o[V];
    value(g, o);
#pragma unroll
    for (int i = 0; i < V; ++i) ss = fmaf(o[i], o[i], ss);
  }
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)H + eps);
  auto finish = [&](int g, const float (&o)[V]) {
    float h[V], wv[V];
    pn_load<float, V>(x + base + (size_t)g * V, h);
    pn_load<TW, V>(w + (size_t)g * V, wv);
#pragma unroll
    for (int i = 0; i < V; ++i) h[i] += mult * (o[i] * inv * wv[i]);
    pn_store<float, V>(x + base + (size_t)g * V, h);
    if (x_act) pn_store<TA, V>(x_act + base + (size_t)g * V, h);
  };
#pragma unroll
  for (int u = 0; u < PN_KEEP; ++u) {
    const int g = threadIdx.x + u * blockDim.x;
    if (g < groups) finish(g, keep[u]);
  }
  for (int g = threadIdx.x + PN_KEEP * blockDim.x; g < groups; g += blockDim.x) {
    float o[V];
    value(g, o);
    finish(g, o);
  }
}

static inline int pn_threads(int groups) {
  int n = (groups + 31) / 32 * 32;
  return n < 32 ? 32 : (n > GLUE_THREADS ? GLUE_THREADS : n);
}

// y1 may be null (then s1 is not read); x_act may be null
RLLM_EXPORT int rllm_postnorm_add(float* x, const void* y0, const void* y1, float s0, float s1, const void* w, float eps,
                                  float mult, void* x_act, int T, int H, int act_dtype, int w_dtype,
                                  cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H <= 0 || !x || !y0 || !w) return RLLM_E_BADARG;
  const bool wide = H % 4 == 0 && (((uintptr_t)x | (uintptr_t)y0 | (uintptr_t)y1 | (uintptr_t)w | (uintptr_t)x_act) & 15) == 0;
#define PN_GO(TA, TW, V)                                                                                          \
  rllm_launch_pdl(postnorm_add_kernel<TA, TW, V>, dim3(T), dim3(pn_threads(H / V)), (size_t)0, stream, x,         \
                  (const TA*)y0, (const TA*)y1, s0, s1, (const TW*)w, eps, mult, (TA*)x_act, H)
  RLLM_DISPATCH_DTYPE(act_dtype, TA_, RLLM_DISPATCH_DTYPE(w_dtype, TW_, {
    if (wide) PN_GO(TA_, TW_, 4); else PN_GO(TA_, TW_, 1);
  }));
#undef PN_GO
  RLLM_LAUNCH_CHECK();
  return 0;
}

__global__ void __launch_bounds__(256) activation_rows_kernel(const float* x, bf16* out, long long n) {
  pdl_wait();
  pdl_launch();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i < n) out[i] = from_f32<bf16>(x[i]);
}
RLLM_EXPORT int rllm_activation_rows(const float* x, void* out, long long n, cudaStream_t stream) {
  if (n <= 0) return 0;
  rllm_launch_pdl(activation_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), (size_t)0, stream, x, (bf16*)out, n);
  RLLM_LAUNCH_CHECK();
  return 0;
}

template <typename T>
__global__ void __launch_bounds__(256) scaled_sum2_kernel(const T* a, const T* b, float sa, float sb, T* out, long long n) {
  pdl_wait();
  pdl_launch();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i < n) out[i] = from_f32<T>(fmaf(sb, to_f32(b[i]), sa * to_f32(a[i])));
}
RLLM_EXPORT int rllm_scaled_sum2(const void* a, const void* b, float sa, float sb, void* out, int dtype, long long n,
                                 cudaStream_t stream) {
  if (n <= 0) return 0;
  RLLM_DISPATCH_DTYPE(dtype, TT,
    (rllm_launch_pdl(scaled_sum2_kernel<TT>, dim3((unsigned)((n + 255) / 256)), dim3(256), (size_t)0, stream, (const TT*)a,
                     (const TT*)b, sa, sb, (TT*)out, n)));
  RLLM_LAUNCH_CHECK();
  return 0;
}
