// The step ahead of attention whose heads' scores are mixed ("talking heads", ahead of the softmax):
//
//   s_h(i, j) = scale * sum_g talk[h, g] q_g(i) . k_(g / per)(j),      per = query heads a kv head
//
// The mixture moves to the queries: with q'_h = [sum over the heads g of kv head 0 of talk[h, g] q_g | ... | the same
// for the last kv head] and the token's key row [k_0 | k_1 | ... ], s_h = scale * q'_h(i) . row(j).  A token so has
// ONE key row that all heads read, and head h its own values.  From a token's projections [q | k | v] the kernel makes
//
//   q' (T x H rows of dkp, zeros behind the nkv * dk values) from the queries with their biases, rotated, in float32
//   until the one rounding at the end; the key row (biases, rotation) and the value row (biases; each head's dv values
//   in dvp places, zeros behind them) in the token's place of its cache page; the values optionally mixed with another
//   layer's of the same token, v <- (1 - lambda) v + lambda (v_other + its bias).
#include "common.cuh"
#include <math.h>

#define TH_PER 8                 // query heads a kv head that the quick form of the mixture takes

__device__ __forceinline__ void th_store4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void th_store4(bf16* p, float4 v) {
  uint2 r;
  *(__nv_bfloat162*)&r.x = __floats2bfloat162_rn(v.x, v.y);
  *(__nv_bfloat162*)&r.y = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = r;
}

template <typename T>
__global__ void __launch_bounds__(256)
talking_prep_kernel(const T* qkv, int stride, const int* positions, const int* token_seq, const float* bias,
                    const float* talk, const double* inv_freq, int rd, const T* v_other, int other_stride,
                    const float* other_bias, const float* lambda, const int* block_table, int max_blocks, T* kcache,
                    T* vcache, int page_size, int num_pages, int nq, int nkv, int dk, int dv, int dkp, int dvp, T* q_out,
                    int* err) {
  extern __shared__ __align__(16) float th_smem[];
  float* qs = th_smem;                       // [nq][dk]: rotated queries
  float* tk = qs + nq * dk;                  // [nq][nq]
  float* cs = tk + nq * nq;                  // [rd]: cosines, sines
  const int half = rd >> 1;
  for (int e = threadIdx.x; e < nq * nq; e += blockDim.x) tk[e] = talk[e];
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x, pos = positions[t];
  const T* row = qkv + (size_t)t * stride;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float c, s;
    if (sizeof(T) == 4) {
      double sd, cd;
      sincos((double)pos * inv_freq[i], &sd, &cd);
      c = (float)cd; s = (float)sd;
    } else {
      rope_cos_sin(pos, inv_freq[i], &c, &s);
    }
    cs[i] = c;
    cs[half + i] = s;
  }
  const int blk = pos / page_size;
  const int page = blk < max_blocks ? block_table[(size_t)token_seq[t] * max_blocks + blk] : -1;
  const bool place = page >= 0 && page < num_pages;
  if (!place && threadIdx.x == 0) atomicOr(err, 2);
  const size_t at = place ? (size_t)page * page_size + pos % page_size : 0;
  __syncthreads();
  T* krow = kcache + at * dkp;
  const int items = dk - half;               // a head's pairs, then the dimensions that do not rotate
  for (int e = threadIdx.x; e < (nq + nkv) * items; e += blockDim.x) {
    const int h = e / items, i = e - h * items;
    const int b = h * dk;
    if (i < half) {
      const float x = to_f32(row[b + i]) + bias[b + i], y = to_f32(row[b + i + half]) + bias[b + i + half];
      const float lo = x * cs[i] - y * cs[half + i], hi = y * cs[i] + x * cs[half + i];
      if (h < nq) { qs[b + i] = lo; qs[b + i + half] = hi; }
      else if (place) { krow[b - nq * dk + i] = from_f32<T>(lo); krow[b - nq * dk + i + half] = from_f32<T>(hi); }
    } else {
      const int j = i + half;
      const float x = to_f32(row[b + j]) + bias[b + j];
      if (h < nq) qs[b + j] = x;
      else if (place) krow[b - nq * dk + j] = from_f32<T>(x);
    }
  }
  if (place) {
    for (int c = nkv * dk + threadIdx.x; c < dkp; c += blockDim.x) krow[c] = from_f32<T>(0.f);
    T* vrow = vcache + at * (size_t)nkv * dvp;
    const int vat = (nq + nkv) * dk;
    const float lam = v_other ? lambda[0] : 0.f;
    for (int e = threadIdx.x; e < nkv * dvp; e += blockDim.x) {
      const int g = e / dvp, c = e - g * dvp;
      float v = 0.f;
      if (c < dv) {
        const int j = g * dv + c;
        v = to_f32(row[vat + j]) + bias[vat + j];
        if (v_other) v = fmaf(1.0f - lam, v, lam * (to_f32(v_other[(size_t)t * other_stride + j]) + other_bias[j]));
      }
      vrow[e] = from_f32<T>(v);
    }
  }
  __syncthreads();
  const int per = nq / nkv;
  T* qo = q_out + (size_t)t * nq * dkp;
  if (per <= TH_PER && (dk & 3) == 0) {
    // four neighbouring places of a kv head's part for a share of the heads: its query heads' values stay in registers
    const int quads = nkv * dk / 4, shares = max(1, (int)blockDim.x / quads);
    for (int e = threadIdx.x; e < quads * shares; e += blockDim.x) {
      const int share = e / quads, c = (e - share * quads) * 4, g = c / dk;
      float4 q[TH_PER];
#pragma unroll
      for (int u = 0; u < TH_PER; ++u)
        if (u < per) q[u] = *(const float4*)&qs[(g * per + u) * dk + c - g * dk];
      for (int h = share; h < nq; h += shares) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < TH_PER; ++u) {
          if (u < per) {
            const float w = tk[h * nq + g * per + u];
            v.x = fmaf(w, q[u].x, v.x); v.y = fmaf(w, q[u].y, v.y); v.z = fmaf(w, q[u].z, v.z); v.w = fmaf(w, q[u].w, v.w);
          }
        }
        th_store4(qo + h * dkp + c, v);
      }
    }
    const int pad = dkp - nkv * dk;
    for (int e = threadIdx.x; e < nq * pad; e += blockDim.x) qo[e / pad * dkp + nkv * dk + e % pad] = from_f32<T>(0.f);
    return;
  }
  for (int e = threadIdx.x; e < nq * dkp; e += blockDim.x) {
    const int h = e / dkp, c = e - h * dkp, g = c / dk, i = c - g * dk;
    float v = 0.f;
    if (g < nkv)
      for (int u = 0; u < per; ++u) v = fmaf(tk[h * nq + g * per + u], qs[(g * per + u) * dk + i], v);
    qo[e] = from_f32<T>(v);
  }
}

// qkv: T rows of [nq dk | nkv dk | nkv dv]; bias float32 over such a row; talk float32 [nq, nq]; caches
// [pages, 1, page_size, dkp] and [pages, 1, page_size, nkv dvp]; q_out [T, nq dkp].  v_other: null, or T rows of
// nkv dv values with row stride other_stride, other_bias float32 [nkv dv], lambda float32 [1].
RLLM_EXPORT int rllm_talking_prep(const void* qkv, int stride, int dtype, const int* positions, const int* token_seq,
                                  const float* bias, const float* talk, const double* inv_freq, int rd,
                                  const void* v_other, int other_stride, const float* other_bias, const float* lambda,
                                  const int* block_table, int max_blocks, void* kcache, void* vcache, int page_size,
                                  int num_pages, int T, int nq, int nkv, int dk, int dv, int dkp, int dvp, void* q_out,
                                  int* err, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (nq <= 0 || nkv <= 0 || nq % nkv || dk <= 0 || dv <= 0 || dkp < nkv * dk || dvp < dv) return RLLM_E_BADARG;
  if (rd < 0 || rd > dk || (rd & 1) || (rd > 0 && !inv_freq) || !bias || !talk || page_size <= 0 || num_pages <= 0 ||
      max_blocks <= 0 || stride < nq * dk + nkv * (dk + dv) || (v_other && (!other_bias || !lambda)))
    return RLLM_E_BADARG;
  const size_t smem = sizeof(float) * ((size_t)nq * dk + (size_t)nq * nq + rd);
  if (smem > 200 * 1024) return RLLM_E_UNSUPPORTED;
  if (dkp % 4 || (((uintptr_t)q_out) & 15)) return RLLM_E_BADARG;
  RLLM_DISPATCH_DTYPE(dtype, TT, {
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(talking_prep_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    rllm_launch_pdl(talking_prep_kernel<TT>, dim3(T), dim3(256), smem, stream, (const TT*)qkv, stride, positions, token_seq,
                    bias, talk, inv_freq, rd, (const TT*)v_other, other_stride, other_bias, lambda, block_table, max_blocks,
                    (TT*)kcache, (TT*)vcache, page_size, num_pages, nq, nkv, dk, dv, dkp, dvp, (TT*)q_out, err);
  });
  RLLM_LAUNCH_CHECK();
  return 0;
}
