// Capped softmax attention with a sink and kept first positions, for portions of prompts with keys and values of 64 or 128
// values: the instantiations with options of the tcgen05 kernel of attention_prefill_tcgen05.cu.
#define DLLM_PREFILL_TCGEN05_OPTIONS
#include "attention_prefill_tcgen05.cu"

// As `dllm_attention_prefill_tcgen05`, with the cap (0: none), the sinks ([heads] or null), the first positions that a
// window keeps, the chunks and a factor of the outputs, whose rows have out_stride values (a multiple of 8).
DLLM_EXPORT int dllm_sink_attention_tcgen05(void* out, int out_stride, const void* q, int tokens, void* cache_base,
                                            long long cache_pages, const int* page_table, int max_pages, int page_size,
                                            int heads, int kv_heads, int head_dim, const int* tile_seq,
                                            const int* tile_first, const int* cu_seqlens, const int* start,
                                            const int* slots, int tiles, float scale, float cap, const float* sinks,
                                            int window, int keep, int chunk, float out_scale, int* status, cudaStream_t stream) {
  if (window < 0 || keep < 0 || chunk < 0) return DLLM_BAD_ARGUMENT;
  if (out_stride < heads * head_dim || (out_stride & 7)) return DLLM_UNSUPPORTED_SIZE;
  const ScoreOptions options = {sinks, cap, window > 0 || chunk > 0 ? keep : 0, head_dim, out_stride, chunk, out_scale};
  return run<true>(out, q, tokens, cache_base, cache_pages, page_table, max_pages, page_size, heads, kv_heads, head_dim,
                   tile_seq, tile_first, cu_seqlens, start, slots, tiles, scale, window, status, options, stream);
}
