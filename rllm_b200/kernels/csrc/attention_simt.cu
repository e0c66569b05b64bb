// Paged causal attention on CUDA cores, for float32 and bfloat16 caches: the
// kernel of the true 32-bit path, and the fallback of the bfloat16 path for
// shapes its tensor-core kernels refuse.  One warp per (query token, query
// head); it serves prompt portions and single decoded tokens alike, since a
// token's keys are read from the cache through the block table either way.
//
// Contract (the reference's intended one, crates/rllm-kernels/src/cuda/
// paged_attention.cu:88-179 for the math; its prefill kernel ignores earlier
// context at :285-286, which this does not): the query at position p of
// sequence s sees keys max(0, p - window + 1) .. p of s (window 0: all keys
// 0 .. p); kv head of query head h is h / (nq / nkv) (:113); scores are
// scaled by `scale`; softmax is online in float32 (:159-169), P.V is
// accumulated in float32 and divided by the sum once (:173-178).
//
// Options beyond that contract (each off at 0 / null):
//   keep_first  with a window: keys 0 .. keep_first - 1 stay visible however far back they lie;
//   chunk       the query sees only keys of its own chunk, floor(j / chunk) == floor(p / chunk);
//   softcap     score <- softcap * tanh(score / softcap) after the scaling;
//   sinks       float32 [nq]: exp(sinks[h]) joins the softmax's denominator (no key, no value, unscaled);
//   gate        a row of gate pre-activations beside the token's queries: the result is multiplied by
//               sigmoid(gate[h]) (gate_mode 1, one number a head) or sigmoid(gate[h * dv + i])
//               (gate_mode 2, one a result element);
//   slopes      float32 [nq]: slopes[h] * (p - j) is taken off the score of key j (after scaling and cap):
//               a bias that grows with the distance between query and key.
//
// Keys are walked in groups of 32 aligned to absolute positions, so the
// arithmetic of a row does not depend on how the sequence was cut into steps,
// on the batch around it, or on which pages hold it.
#include "common.cuh"
#include <math.h>

#define ATT_WARPS 4
#define ATT_MAX_D 256

template <typename T> struct Vec8;
template <> struct Vec8<float> {
  static __device__ __forceinline__ void load(const float* p, float* o) {
    float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
    o[0] = a.x; o[1] = a.y; o[2] = a.z; o[3] = a.w; o[4] = b.x; o[5] = b.y; o[6] = b.z; o[7] = b.w;
  }
};
template <> struct Vec8<bf16> {
  static __device__ __forceinline__ void load(const bf16* p, float* o) {
    uint4 a = *(const uint4*)p;
    const __nv_bfloat162* h = (const __nv_bfloat162*)&a;
#pragma unroll
    for (int i = 0; i < 4; ++i) { float2 f = __bfloat1622float2(h[i]); o[2 * i] = f.x; o[2 * i + 1] = f.y; }
  }
};

// d: the size of a query and key head; dv: of a value and output head (they may differ).  VEC: d is a
// multiple of 8 and keys are fetched eight at a time; otherwise one by one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(32 * ATT_WARPS)
attention_simt_kernel(const T* __restrict__ q, int q_stride, T* __restrict__ out,
                      const T* __restrict__ kcache, const T* __restrict__ vcache,
                      const int* __restrict__ block_table, int max_blocks,
                      const int* __restrict__ positions, const int* __restrict__ token_seq, int T_tokens,
                      int nq, int nkv, int d, int dv, int page_size, int num_pages, int window, float scale,
                      int keep_first, int chunk, float softcap, const float* __restrict__ sinks,
                      const T* __restrict__ gate, int gate_stride, int gate_mode,
                      const float* __restrict__ slopes, int shared_keys, int v_ld, int* __restrict__ err) {
  extern __shared__ float qs[];  // [ATT_WARPS][d]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long gw = (long long)blockIdx.x * ATT_WARPS + warp;
  if (gw >= (long long)T_tokens * nq) return;
  const int t = (int)(gw / nq), h = (int)(gw - (long long)t * nq);
  const int kvh = h / (nq / nkv);
  // rows of the caches: which head of a page, how many heads it has, and where a value row of it starts
  const int pg_heads = shared_keys ? 1 : nkv, pg_h = shared_keys ? 0 : kvh;
  const int v_row = shared_keys ? nkv * v_ld : dv, v_off = shared_keys ? kvh * v_ld : 0;
  const int s = token_seq[t];
  const int qpos = positions[t];
  const int kend = qpos + 1;
  int kstart = (window > 0 && qpos - window + 1 > 0) ? qpos - window + 1 : 0;
  if (chunk > 0) kstart = max(kstart, qpos / chunk * chunk);
  // the kept first keys that lie ahead of the recent ones: a range of their own, walked first
  const int kept_end = (window > 0 && keep_first > 0) ? min(min(keep_first, kstart), kend) : 0;
  const int kept_start = (chunk > 0) ? min(qpos / chunk * chunk, kept_end) : 0;
  const float inv_cap = softcap > 0.f ? 1.0f / softcap : 0.f;
  const float slope = slopes ? slopes[h] : 0.f;
  float* myq = qs + warp * d;
  const T* qrow = q + (size_t)t * q_stride + (size_t)h * d;
  for (int i = lane; i < d; i += 32) myq[i] = to_f32(qrow[i]);
  __syncwarp();

  float m = -INFINITY, l = 0.f;
  float acc[ATT_MAX_D / 32];
#pragma unroll
  for (int r = 0; r < ATT_MAX_D / 32; ++r) acc[r] = 0.f;
  const int* bt = block_table + (size_t)s * max_blocks;

  for (int range = 0; range < 2; ++range) {
  const int lo = range == 0 ? kept_start : kstart, hi = range == 0 ? kept_end : kend;
  for (int j0 = (lo / 32) * 32; j0 < hi; j0 += 32) {
    const int j = j0 + lane;
    const bool valid = (j >= lo) && (j < hi);
    float score = -INFINITY;
    int page = -1;
    if (valid) {
      page = bt[j / page_size];
      if (page < 0 || page >= num_pages) {
        atomicOr(err, 4);
        page = -1;
      } else {
        const T* kp = kcache + (((size_t)page * pg_heads + pg_h) * page_size + (j % page_size)) * d;
        float dot = 0.f;
        if (VEC) {
          for (int i = 0; i < d; i += 8) {
            float kv[8];
            Vec8<T>::load(kp + i, kv);
#pragma unroll
            for (int u = 0; u < 8; ++u) dot = fmaf(myq[i + u], kv[u], dot);
          }
        } else {
          for (int i = 0; i < d; ++i) dot = fmaf(myq[i], to_f32(kp[i]), dot);
        }
        score = dot * scale;
        if (softcap > 0.f) score = softcap * tanhf(score * inv_cap);
        if (slopes) score -= slope * (float)(qpos - j);
      }
    }
    const float cmax = warp_max(score);
    const float m_new = fmaxf(m, cmax);
    if (m_new == -INFINITY) continue;  // nothing visible in this group (warp-uniform)
    const float p = (score == -INFINITY) ? 0.f : expf(score - m_new);
    const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);
    l = l * corr + warp_sum(p);
#pragma unroll
    for (int r = 0; r < ATT_MAX_D / 32; ++r) acc[r] *= corr;
    m = m_new;
    const int jn = min(32, hi - j0);
    for (int jj = max(0, lo - j0); jj < jn; ++jj) {
      const float pj = __shfl_sync(0xffffffffu, p, jj);
      const int pg = __shfl_sync(0xffffffffu, page, jj);
      if (pg < 0) continue;
      const T* vp = vcache + (((size_t)pg * pg_heads + pg_h) * page_size + ((j0 + jj) % page_size)) * v_row + v_off;
#pragma unroll
      for (int r = 0; r < ATT_MAX_D / 32; ++r) {
        const int i = lane + 32 * r;
        if (i < dv) acc[r] = fmaf(pj, to_f32(vp[i]), acc[r]);
      }
    }
  }
  }
  if (sinks) {                                   // one more term of the denominator
    const float sk = sinks[h];
    const float m_new = fmaxf(m, sk);
    const float corr = (m == -INFINITY) ? 0.f : expf(m - m_new);
    l = l * corr + expf(sk - m_new);
#pragma unroll
    for (int r = 0; r < ATT_MAX_D / 32; ++r) acc[r] *= corr;
  }
  T* orow = out + ((size_t)t * nq + h) * dv;
  float inv = (l > 0.f) ? 1.0f / l : 0.f;
  const T* grow = gate_mode ? gate + (size_t)t * gate_stride : nullptr;
  if (gate_mode == 1) inv *= 1.0f / (1.0f + expf(-to_f32(grow[h])));
#pragma unroll
  for (int r = 0; r < ATT_MAX_D / 32; ++r) {
    const int i = lane + 32 * r;
    if (i < dv) {
      float v = acc[r] * inv;
      if (gate_mode == 2) v *= 1.0f / (1.0f + expf(-to_f32(grow[(size_t)h * dv + i])));
      orow[i] = from_f32<T>(v);
    }
  }
}

// keys [pages, nkv, page_size, d], values [pages, nkv, page_size, dv], out [T, nq * dv]; with shared_keys: keys
// [pages, 1, page_size, d], values [pages, 1, page_size, nkv * v_ld]
RLLM_EXPORT int rllm_attention_simt_kv(const void* q, int q_stride, void* out, const void* kcache,
                                       const void* vcache, int dtype, const int* block_table,
                                       int max_blocks, const int* positions, const int* token_seq, int T,
                                       int nq, int nkv, int d, int dv, int page_size, int num_pages, int window,
                                       float scale, int keep_first, int chunk, float softcap, const float* sinks,
                                       const void* gate, int gate_stride, int gate_mode, const float* slopes,
                                       int shared_keys, int v_ld, int* err, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv != 0 || d <= 0 || dv <= 0 || page_size <= 0 || num_pages <= 0 ||
      max_blocks <= 0 || window < 0 || keep_first < 0 || chunk < 0 || !(softcap >= 0.f) || gate_mode < 0 ||
      gate_mode > 2 || (gate_mode && !gate) || (shared_keys && v_ld < dv))
    return RLLM_E_BADARG;
  if (dv > ATT_MAX_D || d > 2816) return RLLM_E_UNSUPPORTED;
  const bool vec = d % 8 == 0 && q_stride % 8 == 0 && (((uintptr_t)q | (uintptr_t)kcache) & 31) == 0;
  const long long warps = (long long)T * nq;
  const unsigned blocks = (unsigned)((warps + ATT_WARPS - 1) / ATT_WARPS);
  const size_t smem = (size_t)ATT_WARPS * d * sizeof(float);
#define ATT_GO(VEC_)                                                                                        \
  RLLM_DISPATCH_DTYPE(dtype, T_,                                                                            \
    (attention_simt_kernel<T_, VEC_><<<blocks, 32 * ATT_WARPS, smem, stream>>>(                             \
        (const T_*)q, q_stride, (T_*)out, (const T_*)kcache, (const T_*)vcache, block_table,                \
        max_blocks, positions, token_seq, T, nq, nkv, d, dv, page_size, num_pages, window, scale, keep_first,  \
        chunk, softcap, sinks, (const T_*)gate, gate_stride, gate_mode, slopes, shared_keys, v_ld, err)))
  if (vec) ATT_GO(true); else ATT_GO(false);
#undef ATT_GO
  RLLM_LAUNCH_CHECK();
  return 0;
}

RLLM_EXPORT int rllm_attention_simt(const void* q, int q_stride, void* out, const void* kcache,
                                    const void* vcache, int dtype, const int* block_table,
                                    int max_blocks, const int* positions, const int* token_seq, int T,
                                    int nq, int nkv, int d, int page_size, int num_pages, int window,
                                    float scale, int* err, cudaStream_t stream) {
  if (d % 16 != 0 || d > ATT_MAX_D) return d > 0 ? RLLM_E_UNSUPPORTED : RLLM_E_BADARG;  // head sizes in steps of 16, to 256
  if (q_stride % 8 != 0) return RLLM_E_BADARG;
  return rllm_attention_simt_kv(q, q_stride, out, kcache, vcache, dtype, block_table, max_blocks, positions,
                                token_seq, T, nq, nkv, d, d, page_size, num_pages, window, scale, 0, 0, 0.f, nullptr,
                                nullptr, 0, 0, nullptr, 0, 0, err, stream);
}
