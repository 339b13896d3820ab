// Capped softmax attention with a sink and kept first positions, for single tokens: the instantiations with options of
// the cluster kernel of attention_decode_cluster.cu (bfloat16, keys and values of up to 128 values each, multiples of 8,
// which may differ).
#define DLLM_DECODE_CLUSTER_OPTIONS
#include "attention_decode_cluster.cu"

// out [sequences, out_stride] and q [sequences, heads * dim] bfloat16; shapes as for `dllm_attention_decode_cluster`;
// the outputs are multiplied by out_scale.
DLLM_EXPORT int dllm_sink_attention_decode(void* out, int out_stride, const void* q, void* cache_base,
                                           const int* page_table, int max_pages, int page_size, int heads, int kv_heads,
                                           int dim, int vdim, const int* tok_pos, const int* slots, int sequences,
                                           float scale, float cap, const float* sinks, int window, int keep, int chunk,
                                           float out_scale, int shape,
                                           cudaStream_t stream) {
  if (sequences <= 0) return DLLM_OK;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || window < 0 || keep < 0 || chunk < 0 || shape < -1 || shape >= SHAPES)
    return DLLM_BAD_ARGUMENT;
  if (dim <= 0 || dim > 128 || (dim & 7) || vdim <= 0 || vdim > 128 || (vdim & 7) || page_size != TILE_KEYS ||
      sequences > 65535 || kv_heads > 65535 || out_stride < heads * vdim)
    return DLLM_UNSUPPORTED_SIZE;
  KvLayout cache{cache_base, page_table, max_pages, page_size, kv_heads, dim};
  const ScoreOptions options = {sinks, cap, window > 0 || chunk > 0 ? keep : 0, vdim, out_stride, chunk, out_scale};
  int wider = dim > vdim ? dim : vdim;
  if (wider <= 32)
    return launch_shape<32, true>(shape, out, q, cache, tok_pos, slots, heads, sequences, scale, window, options, stream);
  if (wider <= 64)
    return launch_shape<64, true>(shape, out, q, cache, tok_pos, slots, heads, sequences, scale, window, options, stream);
  return launch_shape<128, true>(shape, out, q, cache, tok_pos, slots, heads, sequences, scale, window, options, stream);
}
