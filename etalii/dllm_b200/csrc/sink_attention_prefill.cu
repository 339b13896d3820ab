// Capped softmax attention with a sink and kept first positions, for portions of prompts: the instantiations with options
// of the mma.sync kernel of attention_prefill.cu (bfloat16, tiles of 64 queries, keys and values of up to 128 values
// each, multiples of 8, which may differ).
#define DLLM_PREFILL_OPTIONS
#include "attention_prefill.cu"

// out [tokens, out_stride] and q [tokens, heads * dim] bfloat16; tiles as for `dllm_attention_prefill`; the outputs are
// multiplied by out_scale.
DLLM_EXPORT int dllm_sink_attention_prefill(void* out, int out_stride, const void* q, void* cache_base,
                                            const int* page_table, int max_pages, int page_size, int heads, int kv_heads,
                                            int dim, int vdim, const int* tile_seq, const int* tile_first,
                                            const int* cu_seqlens, const int* start, const int* slots, int tiles,
                                            float scale, float cap, const float* sinks, int window, int keep, int chunk,
                                            float out_scale,                                            cudaStream_t stream) {
  if (tiles <= 0) return DLLM_OK;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || window < 0 || keep < 0 || chunk < 0) return DLLM_BAD_ARGUMENT;
  if (dim <= 0 || dim > 128 || (dim & 7) || vdim <= 0 || vdim > 128 || (vdim & 7) || page_size != BN || heads > 65535 ||
      out_stride < heads * vdim || (out_stride & 1))
    return DLLM_UNSUPPORTED_SIZE;
  KvLayout cache{cache_base, page_table, max_pages, page_size, kv_heads, dim};
  const ScoreOptions options = {sinks, cap, window > 0 || chunk > 0 ? keep : 0, vdim, out_stride, chunk, out_scale};
  int wider = dim > vdim ? dim : vdim;
  if (wider <= 32)
    return launch<32, true>(out, q, cache, tile_seq, tile_first, cu_seqlens, start, slots, tiles, heads, scale, window,
                            options, stream);
  if (wider <= 64)
    return launch<64, true>(out, q, cache, tile_seq, tile_first, cu_seqlens, start, slots, tiles, heads, scale, window,
                            options, stream);
  return launch<128, true>(out, q, cache, tile_seq, tile_first, cu_seqlens, start, slots, tiles, heads, scale, window,
                           options, stream);
}
