// The state-space recurrence of Mamba-2 (one scalar decay per head and token).  Per head, with B and C of its
// group (size N) and values x of size P:
//
//   dt = softplus(r_t + dt_bias);   S_t = exp(-exp(a_log) dt) S_(t-1) + dt B_t x_t^T   [N, P]
//   y_t = S_t^T C_t + d x_t
//
// S lives in float32 in the request's state slot [heads][N][P], starts at zero and is carried from step to step.
// This is the linear-attention recurrence with q = C, k = B, v = x and factors per token: the kernels are
// lightning attention's (lightning_walk.cuh; lightning_mma.cuh for long bfloat16 portions) with STEPS on.
//
//   ssd_scan                    the recurrence; long portions as chunks of 64 side by side
//   silu_gated_group_rmsnorm    y * silu(z), each of `groups` equal parts of the row over its own root mean
//                               square (eps inside the root), times a weight: one block a (token, group)
#include "lightning_walk.cuh"
#include "lightning_mma.cuh"

RLLM_EXPORT int rllm_ssd_chunk() { return LT_CHUNK; }

// RLLM_SSD=simt keeps the chunk passes on the CUDA cores (for tests and comparisons)
static inline bool ssd_mma_disabled() {
  static int off = -1;
  if (off < 0) { const char* e = getenv("RLLM_SSD"); off = (e && e[0] == 's') ? 1 : 0; }
  return off == 1;
}

// xbc: rows of [x: heads * P | B: groups * N | C: groups * N] with row stride `stride`.  max_chunks 0: the plain
// walk.  > 0: ceil(longest portion / LT_CHUNK); work then holds num_seqs * max_chunks * heads * N * P floats and
// chunk_dt num_seqs * max_chunks * heads.
RLLM_EXPORT int rllm_ssd_scan(const void* xbc, int stride, int dtype, const float* dt, const float* dt_bias,
                              const float* a_log, const float* skip, float* state, float* work, float* chunk_dt,
                              const int* q_start, const int* slots, int num_slots, int num_seqs, int max_chunks,
                              float* out, int heads, int groups, int N, int P, int* err, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups || N <= 0 || P <= 0 || num_slots <= 0 || max_chunks < 0) return RLLM_E_BADARG;
  if (stride < heads * P + 2 * groups * N || (max_chunks > 0 && (!work || !chunk_dt))) return RLLM_E_BADARG;
  if (N > 256 || (long long)num_seqs * (max_chunks > 0 ? max_chunks : 1) > 65535) return RLLM_E_UNSUPPORTED;
  static_assert(LT_CHUNK == LTC_CHUNK, "the chain kernel serves both forms of the chunk passes");
  const LtSteps steps{dt, dt_bias, a_log, skip, chunk_dt, heads / groups};
  if (dtype == RLLM_DT_BF16 && max_chunks > 0 && !ssd_mma_disabled() && N <= 128 && P <= 128) {
    const bf16* x = (const bf16*)xbc;
    const bf16 *B = x + (size_t)heads * P, *C = B + (size_t)groups * N;
    auto chain = [&]() {
      rllm_launch_pdl(lightning_chain_kernel<true>, dim3(heads, num_seqs, (N * P + 255) / 256), dim3(256), (size_t)0, stream,
                      (const float*)nullptr, steps, state, work, q_start, slots, num_slots, max_chunks, heads, N, P);
    };
#define SSD_GO(D_, DV_)                                                                                            \
  ltc_launch<D_, DV_, true>(C, B, x, stride, nullptr, steps, work, q_start, num_seqs, max_chunks, out, heads, N, P, \
                            stream, chain)
    if (N <= 64) { if (P <= 64) SSD_GO(64, 64); else SSD_GO(64, 128); }
    else { if (P <= 64) SSD_GO(128, 64); else SSD_GO(128, 128); }
#undef SSD_GO
    RLLM_LAUNCH_CHECK();
    return 0;
  }
  RLLM_DISPATCH_DTYPE(dtype, TT, {
    const TT* x = (const TT*)xbc;
    const TT* B = x + (size_t)heads * P;
    const TT* C = B + (size_t)groups * N;
    lightning_walk<TT, true>(C, B, x, stride, nullptr, steps, state, work, q_start, slots, num_slots, num_seqs, max_chunks,
                             out, heads, N, P, err, stream);
  });
  RLLM_LAUNCH_CHECK();
  return 0;
}

template <typename T>
__global__ void __launch_bounds__(256)
silu_gated_group_rmsnorm_kernel(const float* y, const T* z, int z_stride, const float* w, T* out, int E, int size,
                                float eps) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch();
  const size_t base = (size_t)blockIdx.x * E + (size_t)blockIdx.y * size;
  const T* zr = z + (size_t)blockIdx.x * z_stride + (size_t)blockIdx.y * size;
  const float* wr = w + (size_t)blockIdx.y * size;
  constexpr int KEEP = 16;                     // gated values a thread keeps for the second pass
  float v[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int i = threadIdx.x + u * blockDim.x;
    v[u] = 0.f;
    if (i < size) v[u] = y[base + i] * lt_silu(to_f32(zr[i]));
    ss = fmaf(v[u], v[u], ss);
  }
  for (int i = threadIdx.x + KEEP * blockDim.x; i < size; i += blockDim.x) {
    const float x = y[base + i] * lt_silu(to_f32(zr[i]));
    ss = fmaf(x, x, ss);
  }
  ss = block_sum(ss, red);
  const float r = 1.0f / sqrtf(ss / (float)size + eps);
#pragma unroll
  for (int u = 0; u < KEEP; ++u) {
    const int i = threadIdx.x + u * blockDim.x;
    if (i < size) out[base + i] = from_f32<T>(v[u] * r * wr[i]);
  }
  for (int i = threadIdx.x + KEEP * blockDim.x; i < size; i += blockDim.x)
    out[base + i] = from_f32<T>(y[base + i] * lt_silu(to_f32(zr[i])) * r * wr[i]);
}

RLLM_EXPORT int rllm_silu_gated_group_rmsnorm(const float* y, const void* z, int z_stride, const float* w, void* out,
                                              int dtype, int T, int E, int groups, float eps, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (E <= 0 || groups <= 0 || E % groups || z_stride < E) return RLLM_E_BADARG;
  if (groups > 65535) return RLLM_E_UNSUPPORTED;
  const int size = E / groups;
  int threads = (size / 8 + 31) / 32 * 32;
  threads = threads < 32 ? 32 : (threads > 256 ? 256 : threads);
  RLLM_DISPATCH_DTYPE(dtype, TT,
    (rllm_launch_pdl(silu_gated_group_rmsnorm_kernel<TT>, dim3(T, groups), dim3(threads), (size_t)0, stream, y,
                     (const TT*)z, z_stride, w, (TT*)out, E, size, eps)));
  RLLM_LAUNCH_CHECK();
  return 0;
}
