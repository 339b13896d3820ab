// Softmax attention over the paged cache with capped scores, a sink and a window that keeps a sequence's first positions:
// position i sees j <= i with i - j < window, or those of its own chunk of `chunk` positions, and the first `keep` positions
// at any distance; a visible key's score is
// cap tanh(q . k * scale / cap) (cap 0: q . k * scale); the softmax's denominator also holds exp(sink_h), a number per
// head that has no key and no value. Keys have `dim` values, values `vdim`.
//
//   sink_attention:        the general kernel, either cache type and every size up to 256: a warp per (token, query
//                          head) walks the tiles of 32 keys the token sees, one key a lane for the scores, one value
//                          place a lane for the weighted sum, a running maximum and sum; float32 arithmetic. A result
//                          depends only on the token's own query and the keys it sees.
//   sink_attention_split:  the same for steps of few tokens: the warps of a block share one (token, head), each walks
//                          every WARPS-th tile, and their partial results are combined in warp order.
//
// Cache entry: [page][ keys: kv_head, row, dim | values: kv_head, row, vdim ] (wide_kv.cuh).
#include "wide_kv.cuh"

namespace {
constexpr int WARPS = 4, SPLIT_WARPS = 16, TILE = 32, MAX_DIM = 256;
constexpr int PLACES = MAX_DIM / 32;  // value places a lane owns

struct SinkArgs {
  const void* q;       // [tokens, heads * dim] in the cache's type
  void* out;           // [tokens, out_stride] in the cache's type; `fill` zeros behind heads * vdim
  int out_stride;
  WideKv cache;
  const float* sinks;  // [heads] or null
  const int* tok_seq;
  const int* tok_pos;
  const int* slots;
  int tokens, heads, fill, window, keep, chunk;
  float scale, cap, out_scale;
};

__device__ __forceinline__ float dot_piece(const float* q, const float* k) {
  float4 v = *reinterpret_cast<const float4*>(k);
  return fmaf(q[3], v.w, fmaf(q[2], v.z, fmaf(q[1], v.y, q[0] * v.x)));
}
__device__ __forceinline__ float dot_piece(const float* q, const __nv_bfloat16* k) {
  uint4 raw = *reinterpret_cast<const uint4*>(k);
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    float2 x = __bfloat1622float2(p[i]);
    s = fmaf(q[2 * i], x.x, s);
    s = fmaf(q[2 * i + 1], x.y, s);
  }
  return s;
}

struct Running {
  float m, l, acc[PLACES];
  __device__ __forceinline__ void clear() {
    m = -INFINITY;
    l = 0.f;
#pragma unroll
    for (int i = 0; i < PLACES; ++i) acc[i] = 0.f;
  }
};

template <typename T>
__device__ __forceinline__ void one_tile(Running& r, const SinkArgs& a, const float* q_s, const int* pages, int g, int pos,
                                         int first, int j0, int lane) {
  constexpr int N = 16 / sizeof(T);
  const T* base = (const T*)a.cache.base;
  const int dim = a.cache.key_dim, vdim = a.cache.value_dim, ps = a.cache.page_size;
  const int j = j0 + lane;
  const bool seen = j <= pos && (j >= first || j < a.keep);
  const int page = seen ? pages[j / ps] : 0;
  float s = -INFINITY;
  if (seen) {
    const T* key = base + key_at(a.cache, page, g, j % ps);
    float dot = 0.f;
    if (dim % N == 0)
      for (int d = 0; d < dim; d += N) dot += dot_piece(q_s + d, key + d);
    else
      for (int d = 0; d < dim; ++d) dot = fmaf(q_s[d], to_float(key[d]), dot);
    s = dot * a.scale;
    if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
  }
  float m = fmaxf(r.m, warp_max(s));
  if (m == -INFINITY) return;  // (nothing seen so far)
  float p = seen ? expf(s - m) : 0.f, keep = expf(r.m - m);
  r.l = r.l * keep + warp_sum(p);
  r.m = m;
#pragma unroll
  for (int i = 0; i < PLACES; ++i) r.acc[i] *= keep;
  for (unsigned left = __ballot_sync(0xffffffffu, seen); left != 0; left &= left - 1) {
    int jj = __ffs(left) - 1;
    float pj = __shfl_sync(0xffffffffu, p, jj);
    int pg = __shfl_sync(0xffffffffu, page, jj);
    const T* value = base + value_at(a.cache, pg, g, (j0 + jj) % ps);
#pragma unroll
    for (int i = 0; i < PLACES; ++i)
      if (lane + 32 * i < vdim) r.acc[i] = fmaf(pj, to_float(value[lane + 32 * i]), r.acc[i]);
  }
}

template <typename T>
__device__ __forceinline__ void finish(Running& r, const SinkArgs& a, int t, int h, int lane) {
  const int vdim = a.cache.value_dim;
  float factor = 1.f;
  if (a.sinks != nullptr) {  // one more term of the denominator
    float sink = a.sinks[h], m = fmaxf(r.m, sink);
    factor = expf(r.m - m);
    r.l = r.l * factor + expf(sink - m);
  }
  factor *= a.out_scale / r.l;
  T* row = (T*)a.out + (size_t)t * a.out_stride;
#pragma unroll
  for (int i = 0; i < PLACES; ++i)
    if (lane + 32 * i < vdim) row[(size_t)h * vdim + lane + 32 * i] = from_float<T>(r.acc[i] * factor);
  if (h == a.heads - 1)
    for (int i = lane; i < a.fill; i += 32) row[a.heads * vdim + i] = from_float<T>(0.f);
}

template <typename T>
__global__ void __launch_bounds__(WARPS * 32) sink_attention_kernel(SinkArgs a) {
  __shared__ __align__(16) float q_s[WARPS][MAX_DIM];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long long item = (long long)blockIdx.x * WARPS + warp;
  if (item >= (long long)a.tokens * a.heads) return;
  const int t = (int)(item / a.heads), h = (int)(item % a.heads), g = h / (a.heads / a.cache.kv_heads);
  const int pos = a.tok_pos[t], dim = a.cache.key_dim;
  const int* pages = a.cache.page_table + (size_t)a.slots[a.tok_seq[t]] * a.cache.max_pages;
  const T* q = (const T*)a.q + (size_t)item * dim;
  for (int d = lane; d < dim; d += 32) q_s[warp][d] = to_float(q[d]);
  __syncwarp();
  Running r;
  r.clear();
  const KeyWalk walk(pos, pos, a.window, a.keep, TILE, a.chunk);
  const int first = first_visible(pos, a.chunk, a.window);
  for (int i = 0; i < walk.count; ++i) one_tile<T>(r, a, q_s[warp], pages, g, pos, first, walk.tile(i) * TILE, lane);
  finish<T>(r, a, t, h, lane);
}

template <typename T>
__global__ void __launch_bounds__(SPLIT_WARPS * 32) sink_attention_split_kernel(SinkArgs a) {
  __shared__ __align__(16) float q_s[MAX_DIM];
  __shared__ float part_ml[SPLIT_WARPS][2];
  extern __shared__ float part_acc[];  // [SPLIT_WARPS][vdim]
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x / a.heads, h = blockIdx.x % a.heads, g = h / (a.heads / a.cache.kv_heads);
  const int pos = a.tok_pos[t], dim = a.cache.key_dim, vdim = a.cache.value_dim;
  const int* pages = a.cache.page_table + (size_t)a.slots[a.tok_seq[t]] * a.cache.max_pages;
  const T* q = (const T*)a.q + (size_t)blockIdx.x * dim;
  for (int d = threadIdx.x; d < dim; d += blockDim.x) q_s[d] = to_float(q[d]);
  __syncthreads();
  Running r;
  r.clear();
  const KeyWalk walk(pos, pos, a.window, a.keep, TILE, a.chunk);
  const int first = first_visible(pos, a.chunk, a.window);
  for (int i = warp; i < walk.count; i += SPLIT_WARPS) one_tile<T>(r, a, q_s, pages, g, pos, first, walk.tile(i) * TILE, lane);
  if (lane == 0) { part_ml[warp][0] = r.m; part_ml[warp][1] = r.l; }
#pragma unroll
  for (int i = 0; i < PLACES; ++i)
    if (lane + 32 * i < vdim) part_acc[(size_t)warp * vdim + lane + 32 * i] = r.acc[i];
  __syncthreads();
  if (warp != 0) return;
  Running total;
  total.clear();
  for (int w = 0; w < SPLIT_WARPS; ++w) total.m = fmaxf(total.m, part_ml[w][0]);
  for (int w = 0; w < SPLIT_WARPS; ++w) {
    if (part_ml[w][0] == -INFINITY) continue;  // (a warp without a visible key)
    float f = expf(part_ml[w][0] - total.m);
    total.l = fmaf(part_ml[w][1], f, total.l);
#pragma unroll
    for (int i = 0; i < PLACES; ++i)
      if (lane + 32 * i < vdim) total.acc[i] = fmaf(part_acc[(size_t)w * vdim + lane + 32 * i], f, total.acc[i]);
  }
  finish<T>(total, a, t, h, lane);
}

template <typename T>
int launch(const SinkArgs& a, int split, cudaStream_t stream) {
  long long items = (long long)a.tokens * a.heads;
  if (split)
    return dllm_launch_pdl(sink_attention_split_kernel<T>, dim3((unsigned)items), dim3(SPLIT_WARPS * 32),
                           (size_t)SPLIT_WARPS * a.cache.value_dim * sizeof(float), stream, a);
  return dllm_launch_pdl(sink_attention_kernel<T>, dim3((unsigned)((items + WARPS - 1) / WARPS)), dim3(WARPS * 32), 0,
                         stream, a);
}
}  // namespace

// q [tokens, heads * dim] and out [tokens, out_stride] in the cache's type; sinks [heads] float32 or null; window 0 and
// chunk 0: all positions; cap 0: scores as they are; the outputs are multiplied by out_scale, `fill` zeros
// follow a row's. `split` != 0: a block of sixteen warps per (token, head) instead of a warp.
DLLM_EXPORT int dllm_sink_attention(const void* q, void* out, int out_stride, void* cache_base, const int* page_table,
                                    int max_pages, int page_size, int heads, int kv_heads, int dim, int vdim,
                                    const float* sinks, const int* tok_seq, const int* tok_pos, const int* slots,
                                    int tokens, float scale, float cap, int window, int keep, int chunk, float out_scale,
                                    int fill, int split, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return DLLM_OK;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || dim > MAX_DIM || vdim <= 0 || vdim > MAX_DIM ||
      page_size <= 0 || page_size % TILE || window < 0 || keep < 0 || chunk < 0 || fill < 0 ||
      out_stride < heads * vdim + fill)
    return DLLM_UNSUPPORTED_SIZE;
  if (!q || !out || !cache_base || !page_table || !tok_seq || !tok_pos || !slots) return DLLM_BAD_ARGUMENT;
  SinkArgs a = {q, out, out_stride, {cache_base, page_table, max_pages, page_size, kv_heads, dim, vdim}, sinks, tok_seq,
                tok_pos, slots, tokens, heads, fill, window, keep, chunk, scale, cap, out_scale};
  if (dtype == DLLM_F32) return launch<float>(a, split, stream);
  if (dtype == DLLM_BF16) return launch<__nv_bfloat16>(a, split, stream);
  return DLLM_BAD_ARGUMENT;
}
