// Linear attention with a fixed decay per head ("lightning attention"):
//   q_t = silu(a_q), k_t = silu(a_k) [heads, d],  v_t = silu(a_v) [heads, dv]   (a_*: the token's projections)
//   S_t = lambda_h S_{t-1} + k_t v_t^T        (S: [d, dv] per head, float32, per request)
//   o_t = S_t^T q_t                            (no other scale)
// The state lives in the request's state slot [heads, d, dv] and is carried from step to step.
// Activations, state, products and sums are float32; the output is float32 (a norm reads it).
//
// A block owns a head of a sequence (and a range of value columns); a thread keeps an 8 x 8 tile of S in
// registers, eight rows of the head's d (its "slice") by eight value columns.  The block walks the tokens
// in order, eight at a time (their activated q, k and v rows are staged in shared memory); a token's
// output column is the sum over the slices, taken with shuffles inside the warp.  So a token's result
// does not depend on how the sequence was cut or on the batch.
//
// Long portions: the tokens of a sequence in this step are cut into chunks of LT_CHUNK that run
// side by side.  The recurrence is linear in S: first every chunk computes its end state from a
// zero start, then a small kernel chains them (start of chunk c+1 = lambda^len(c) * start of
// chunk c + end-from-zero of chunk c, in order, and the sequence's new state), then every chunk
// walks its tokens from its start.  Results differ from the plain walk by rounding only.
#include "lightning_walk.cuh"
#include "lightning_mma.cuh"

// max_chunks 0: the plain walk.  > 0: ceil(longest portion / LT_CHUNK); work then holds
// num_seqs * max_chunks * heads * d * dv floats.
RLLM_EXPORT int rllm_lightning_chunk() { return LT_CHUNK; }

// RLLM_LIGHTNING=simt keeps the chunk passes on the CUDA cores (for tests and comparisons)
static inline bool lightning_mma_disabled() {
  static int off = -1;
  if (off < 0) { const char* e = getenv("RLLM_LIGHTNING"); off = (e && e[0] == 's') ? 1 : 0; }
  return off == 1;
}

RLLM_EXPORT int rllm_lightning_scan(const void* q, const void* k, const void* v, int stride, int dtype,
                                    const float* decay, float* state, float* work, const int* q_start,
                                    const int* slots, int num_slots, int num_seqs, int max_chunks, float* out,
                                    int heads, int d, int dv, int* err, cudaStream_t stream) {
  if (num_seqs <= 0) return 0;
  if (heads <= 0 || d <= 0 || dv <= 0 || num_slots <= 0 || max_chunks < 0) return RLLM_E_BADARG;
  if (max_chunks > 0 && !work) return RLLM_E_BADARG;
  if (d > 256) return RLLM_E_UNSUPPORTED;               // 32 slices of eight rows: the partners of a sum are one warp
  if ((long long)num_seqs * (max_chunks > 0 ? max_chunks : 1) > 65535) return RLLM_E_UNSUPPORTED;
  static_assert(LT_CHUNK == LTC_CHUNK, "the chain kernel serves both forms of the chunk passes");
  if (dtype == RLLM_DT_BF16 && max_chunks > 0 && !lightning_mma_disabled() && stride % 2 == 0) {
    // long portions of bfloat16 activations: the chunk passes on the tensor cores, where the head's sizes are built
    auto chain = [&]() {
      rllm_launch_pdl(lightning_chain_kernel<false>, dim3(heads, num_seqs, (d * dv + 255) / 256), dim3(256), (size_t)0, stream,
                      decay, LtSteps{}, state, work, q_start, slots, num_slots, max_chunks, heads, d, dv);
    };
    bool done = false;
#define LTC_GO(D_, DV_)                                                                                          \
  if (!done && d == D_ && dv == DV_)                                                                             \
    done = ltc_launch<D_, DV_, false>((const bf16*)q, (const bf16*)k, (const bf16*)v, stride, decay, LtSteps{}, work, q_start,     \
                               num_seqs, max_chunks, out, heads, d, dv, stream, chain)
    LTC_GO(32, 64); LTC_GO(32, 128); LTC_GO(64, 64); LTC_GO(64, 128); LTC_GO(128, 64); LTC_GO(128, 128);
#undef LTC_GO
    if (done) {
      RLLM_LAUNCH_CHECK();
      return 0;
    }
  }
  RLLM_DISPATCH_DTYPE(dtype, TT,
    (lightning_walk<TT, false>((const TT*)q, (const TT*)k, (const TT*)v, stride, decay, LtSteps{}, state, work, q_start,
                               slots, num_slots, num_seqs, max_chunks, out, heads, d, dv, err, stream)));
  RLLM_LAUNCH_CHECK();
  return 0;
}
