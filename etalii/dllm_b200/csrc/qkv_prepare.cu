// From a token's projected float32 row [ ... q (heads x dim) ... k (kv_heads x dim) ... v (kv_heads x vdim) ... ] to what
// attention reads: biases, an RMS norm of every query and key head (one weight of `dim` values for all heads), rotary
// positions on the first `rotary_dim` dimensions (dimension i turns with i + rotary_dim / 2), and for values the mixing
// with another layer's values of the same token, v <- (1 - share) v + share first. Queries go to their buffer, keys and
// values into the token's place in the cache. Every step is optional; all arithmetic is float32, rounded once on the way
// out.
//
// A warp owns one head of one token (a query head, a key head or a value head): its values lie in the lanes' registers,
// value d in lane d % 32, and meet their rotary partners in shared memory.
//
// Cache entry: [page][ keys: kv_head, row, dim | values: kv_head, row, vdim ] (wide_kv.cuh).
#include "wide_kv.cuh"

namespace {
constexpr int WARPS = 4, MAX_DIM = 256, PLACES = MAX_DIM / 32;

struct PrepareArgs {
  const float* rows;
  int stride, q_at, k_at, v_at, heads;
  const float* q_bias;    // [heads * dim], [kv_heads * dim], [kv_heads * vdim], each or null
  const float* k_bias;
  const float* v_bias;
  const float* q_weight;  // [dim] or null (no norm)
  const float* k_weight;
  float eps;
  const float2* table;    // [positions][rotary_dim / 2] (cos, sin) or null
  int rotary_dim;
  float* first;           // [tokens][kv_heads * vdim]: null, written (keeps != 0) or mixed in
  int keeps;
  float share;
  void* q_out;            // [tokens][heads * dim] in the cache's type
  WideKv cache;
  const int* tok_seq;
  const int* tok_pos;
  const int* slots;
  int tokens, write_cache;
};

template <typename T>
__global__ void __launch_bounds__(WARPS * 32) qkv_prepare_kernel(PrepareArgs a) {
  __shared__ float head_s[WARPS][MAX_DIM];
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t = blockIdx.x, groups = a.cache.kv_heads, dim = a.cache.key_dim, vdim = a.cache.value_dim;
  const int unit = blockIdx.y * WARPS + warp;  // query heads, then key heads, then value heads
  if (unit >= a.heads + (a.write_cache ? 2 * groups : 0)) return;
  const float* row = a.rows + (size_t)t * a.stride;
  const int pos = a.tok_pos[t];
  const bool query = unit < a.heads;
  T* base = (T*)a.cache.base;
  int page = 0, at = 0;
  if (!query) {
    page = a.cache.page_table[(size_t)a.slots[a.tok_seq[t]] * a.cache.max_pages + pos / a.cache.page_size];
    at = pos % a.cache.page_size;
  }
  if (unit >= a.heads + groups) {  // values
    const int g = unit - a.heads - groups;
    T* dst = base + value_at(a.cache, page, g, at);
#pragma unroll
    for (int i = 0; i < PLACES; ++i) {
      const int d = lane + 32 * i;
      if (d >= vdim) break;
      float v = row[a.v_at + g * vdim + d];
      if (a.v_bias != nullptr) v += a.v_bias[g * vdim + d];
      if (a.first != nullptr) {
        float* kept = a.first + (size_t)t * groups * vdim + g * vdim + d;
        if (a.keeps) *kept = v;
        else v = fmaf(a.share, *kept, (1.0f - a.share) * v);
      }
      dst[d] = from_float<T>(v);
    }
    return;
  }
  const int h = query ? unit : unit - a.heads;
  const float* src = row + (query ? a.q_at : a.k_at) + h * dim;
  const float* bias = query ? a.q_bias : a.k_bias;
  const float* weight = query ? a.q_weight : a.k_weight;
  float x[PLACES], sum = 0.f;
#pragma unroll
  for (int i = 0; i < PLACES; ++i) {
    const int d = lane + 32 * i;
    x[i] = d < dim ? src[d] + (bias != nullptr ? bias[h * dim + d] : 0.f) : 0.f;
    sum = fmaf(x[i], x[i], sum);
  }
  if (weight != nullptr) {
    const float inv = 1.0f / sqrtf(warp_sum(sum) / (float)dim + a.eps);
#pragma unroll
    for (int i = 0; i < PLACES; ++i)
      if (lane + 32 * i < dim) x[i] *= inv * weight[lane + 32 * i];
  }
  if (a.table != nullptr) {
    const int half = a.rotary_dim >> 1;
#pragma unroll
    for (int i = 0; i < PLACES; ++i)
      if (lane + 32 * i < a.rotary_dim) head_s[warp][lane + 32 * i] = x[i];
    __syncwarp();
    const float2* angles = a.table + (size_t)pos * half;
#pragma unroll
    for (int i = 0; i < PLACES; ++i) {
      const int d = lane + 32 * i;
      if (d >= a.rotary_dim) break;
      if (d < half) {
        float2 c = angles[d];
        x[i] = x[i] * c.x - head_s[warp][d + half] * c.y;
      } else {
        float2 c = angles[d - half];
        x[i] = x[i] * c.x + head_s[warp][d - half] * c.y;
      }
    }
  }
  T* dst = query ? (T*)a.q_out + ((size_t)t * a.heads + h) * dim : base + key_at(a.cache, page, h, at);
#pragma unroll
  for (int i = 0; i < PLACES; ++i)
    if (lane + 32 * i < dim) dst[lane + 32 * i] = from_float<T>(x[i]);
}
}  // namespace

// `first` [tokens][kv_heads * vdim] float32 or null: with `keeps` the values (biases added) are stored there as well as in
// the cache, without it they are mixed with what is stored there. table: [table positions][rotary_dim / 2] (cos, sin).
DLLM_EXPORT int dllm_qkv_prepare(const float* rows, int stride, int q_at, int k_at, int v_at, int heads, int kv_heads,
                                 int dim, int vdim, const float* q_bias, const float* k_bias, const float* v_bias,
                                 const float* q_weight, const float* k_weight, float eps, const float* table,
                                 int rotary_dim, float* first, int keeps, float share, void* q_out, void* cache_base,
                                 const int* page_table, int max_pages, int page_size, const int* tok_seq,
                                 const int* tok_pos, const int* slots, int tokens, int write_cache, int dtype,
                                 cudaStream_t stream) {
  if (tokens <= 0) return DLLM_OK;
  if (heads <= 0 || kv_heads <= 0 || dim <= 0 || dim > MAX_DIM || vdim <= 0 || vdim > MAX_DIM || page_size <= 0 ||
      rotary_dim < 0 || rotary_dim > dim || (rotary_dim & 1) || heads + 2 * kv_heads > 65535 * WARPS)
    return DLLM_UNSUPPORTED_SIZE;
  if (!rows || !q_out || !cache_base || !page_table || !tok_seq || !tok_pos || !slots) return DLLM_BAD_ARGUMENT;
  PrepareArgs a = {rows, stride, q_at, k_at, v_at, heads, q_bias, k_bias, v_bias, q_weight, k_weight, eps,
                   (const float2*)table, rotary_dim, first, keeps, share, q_out,
                   {cache_base, page_table, max_pages, page_size, kv_heads, dim, vdim}, tok_seq, tok_pos, slots, tokens,
                   write_cache};
  const int units = heads + (write_cache ? 2 * kv_heads : 0);
  dim3 grid(tokens, (units + WARPS - 1) / WARPS), block(WARPS * 32);
  if (dtype == DLLM_F32) return dllm_launch_pdl(qkv_prepare_kernel<float>, grid, block, 0, stream, a);
  if (dtype == DLLM_BF16) return dllm_launch_pdl(qkv_prepare_kernel<__nv_bfloat16>, grid, block, 0, stream, a);
  return DLLM_BAD_ARGUMENT;
}
