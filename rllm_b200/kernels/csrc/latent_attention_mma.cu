// Attention over cached latent rows on the tensor cores: the entry point (the kernel is in the header).
#include "latent_attention_mma.cuh"

// work size in floats for a split launch: rows are padded to the row tile the launch will choose
RLLM_EXPORT long long rllm_latent_attention_mma_work(int S, int max_q, int heads, int dv, int nsplit) {
  const long long rows = (long long)max_q * heads;
  const int mt = rows <= 16 ? 1 : (rows <= 32 ? 2 : (dv > 256 ? 2 : 4));
  const int nvt = dv <= 32 ? 1 : (dv <= 64 ? 2 : (dv <= 128 ? 4 : (dv <= 256 ? 8 : 16)));
  const long long padded = (rows + 16 * mt - 1) / (16 * mt) * (16 * mt);
  return (long long)S * padded * nsplit * (32 * nvt + 2);
}

// q [T, heads * dk], out [T, heads * dv], cache [pages, 1, page_size, dk]; sequence s owns tokens
// q_start[s] .. q_start[s+1] and holds seq_lens[s] tokens after this step; max_q: the most tokens a
// sequence brings.  Needs dk % 8 == 0, dv <= min(dk, 512) and 16-byte aligned buffers.
RLLM_EXPORT int rllm_latent_attention_mma(const void* q, void* out, const void* cache, const int* block_table,
                                          int max_blocks, const int* q_start, const int* seq_lens, int S, int max_q,
                                          int heads, int dk, int dv, int page_size, int num_pages, int window,
                                          float scale, const float* sink, int split_keys, int nsplit, float* work,
                                          int* err, cudaStream_t stream) {
  if (S <= 0 || max_q <= 0) return 0;
  if (split_keys > 0 && (split_keys % 64 != 0 || nsplit <= 0 || nsplit > 8192 || work == nullptr)) return RLLM_E_BADARG;
  if (heads <= 0 || dk <= 0 || dv <= 0 || dv > dk || page_size <= 0 || num_pages <= 0 || max_blocks <= 0 ||
      window < 0)
    return RLLM_E_BADARG;
  if (dk % 8 != 0 || dv > 512 || (((uintptr_t)q | (uintptr_t)out | (uintptr_t)cache) & 15) != 0)
    return RLLM_E_UNSUPPORTED;
#define LAM_GO(MT_, NVT_, NW_)                                                                              \
  return lam_launch<MT_, NVT_, NW_>((const bf16*)q, (bf16*)out, (const bf16*)cache, block_table, max_blocks, q_start, \
                               seq_lens, S, max_q, heads, dk, dv, page_size, num_pages, window, scale, sink,   \
                               split_keys, nsplit, work, err, stream)
  // as many row tiles of 16 as the sequences' rows fill, up to what the accumulators leave room for
  const long long rows = (long long)max_q * heads;
  const int mt = rows <= 16 ? 1 : (rows <= 32 ? 2 : 4);
#define LAM_PICK(NVT_, MAXMT_, NW_)                      \
  do {                                                   \
    if (mt == 1) LAM_GO(1, NVT_, NW_);                   \
    if (mt == 2 || MAXMT_ == 2) LAM_GO(2, NVT_, NW_);    \
    LAM_GO(MAXMT_, NVT_, NW_);                           \
  } while (0)
  if (dv <= 32) LAM_PICK(1, 4, 4);
  if (dv <= 64) LAM_PICK(2, 4, 4);
  if (dv <= 128) LAM_PICK(2, 4, 8);
  if (dv <= 256) LAM_PICK(4, 4, 8);
  LAM_PICK(8, 2, 8);
#undef LAM_PICK
#undef LAM_GO
}
