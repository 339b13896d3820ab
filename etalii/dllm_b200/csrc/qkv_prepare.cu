// From a token's projected float32 row [ ... q (heads x dim) ... k (kv_heads x dim) ... v (kv_heads x vdim) ... ] to what
// attention reads: biases, an RMS norm of every query and key head (one weight of `dim` values for all heads), rotary
// positions on the first `rotary_dim` dimensions (dimension i turns with i + rotary_dim / 2), and for values the mixing
// with another layer's values of the same token, v <- (1 - share) v + share first. Queries go to their buffer, keys and
// values into the token's place in the cache. Every step is optional; all arithmetic is float32, rounded once on the way
// out.
//
// A warp owns one head of one token (a query head, a key head or a value head): its values lie in the lanes' registers,
// value d in lane d % 32, and meet their rotary partners in shared memory. Where everything comes in fours (sizes, offsets,
// half the rotated dimensions) and no head is longer than 128, the second kernel gives a head to 8, 16 or 32 lanes with
// four consecutive values each: 16-byte loads, rotary partners by a shuffle.
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
__device__ __forceinline__ void store_four(float* dst, float4 v) { *reinterpret_cast<float4*>(dst) = v; }
__device__ __forceinline__ void store_four(__nv_bfloat16* dst, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
}
__device__ __forceinline__ float4 four(const float* p, int at) {
  return p != nullptr ? *reinterpret_cast<const float4*>(p + at) : make_float4(0.f, 0.f, 0.f, 0.f);
}

template <typename T, int LANES>
__global__ void __launch_bounds__(WARPS * 32) qkv_prepare_fours_kernel(PrepareArgs a) {
  constexpr int PER_BLOCK = WARPS * 32 / LANES;
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x, groups = a.cache.kv_heads, dim = a.cache.key_dim, vdim = a.cache.value_dim;
  const int unit = blockIdx.y * PER_BLOCK + threadIdx.x / LANES, d = 4 * (threadIdx.x % LANES);
  const bool exists = unit < a.heads + (a.write_cache ? 2 * groups : 0);  // (all lanes stay for the shuffles)
  const float* row = a.rows + (size_t)t * a.stride;
  const int pos = a.tok_pos[t];
  const bool query = unit < a.heads, value = unit >= a.heads + groups;
  T* base = (T*)a.cache.base;
  int page = 0, at = 0;
  if (!query) {
    page = a.cache.page_table[(size_t)a.slots[a.tok_seq[t]] * a.cache.max_pages + pos / a.cache.page_size];
    at = pos % a.cache.page_size;
  }
  const int h = query ? unit : value ? unit - a.heads - groups : unit - a.heads;
  const int size = value ? vdim : dim;
  const bool mine = exists && d < size;
  float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
  if (mine) {
    x = four(row, (query ? a.q_at : value ? a.v_at : a.k_at) + h * size + d);
    const float4 b = four(query ? a.q_bias : value ? a.v_bias : a.k_bias, h * size + d);
    x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
  }
  const float* weight = query ? a.q_weight : a.k_weight;
  if (a.q_weight != nullptr || a.k_weight != nullptr) {  // (all lanes take part; a value's sum is not used)
    float sum = fmaf(x.w, x.w, fmaf(x.z, x.z, fmaf(x.y, x.y, x.x * x.x)));
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (mine && !value && weight != nullptr) {
      const float inv = 1.0f / sqrtf(sum / (float)dim + a.eps);
      const float4 w = four(weight, d);
      x.x *= inv * w.x; x.y *= inv * w.y; x.z *= inv * w.z; x.w *= inv * w.w;
    }
  }
  if (a.table != nullptr) {
    const int half = a.rotary_dim >> 1;
    const bool lower = d < half;
    // (a lane outside the rotated places reads some lane of its own head and does not use it)
    const int from = (threadIdx.x & 31 & ~(LANES - 1)) + (((lower ? d + half : d - half) >> 2) & (LANES - 1));
    float4 p;
    p.x = __shfl_sync(0xffffffffu, x.x, from);
    p.y = __shfl_sync(0xffffffffu, x.y, from);
    p.z = __shfl_sync(0xffffffffu, x.z, from);
    p.w = __shfl_sync(0xffffffffu, x.w, from);
    if (mine && !value && d < a.rotary_dim) {
      const float4* angles = reinterpret_cast<const float4*>(a.table + (size_t)pos * half + (lower ? d : d - half));
      const float4 c01 = angles[0], c23 = angles[1];  // (cos, sin) of four pairs
      const float turn = lower ? -1.0f : 1.0f;
      x.x = x.x * c01.x + turn * p.x * c01.y;
      x.y = x.y * c01.z + turn * p.y * c01.w;
      x.z = x.z * c23.x + turn * p.z * c23.y;
      x.w = x.w * c23.z + turn * p.w * c23.w;
    }
  }
  if (!mine) return;
  if (value && a.first != nullptr) {
    float* kept = a.first + (size_t)t * groups * vdim + h * vdim + d;
    if (a.keeps) {
      store_four(kept, x);
    } else {
      const float4 k = four(kept, 0);
      const float own = 1.0f - a.share;
      x.x = fmaf(a.share, k.x, own * x.x); x.y = fmaf(a.share, k.y, own * x.y);
      x.z = fmaf(a.share, k.z, own * x.z); x.w = fmaf(a.share, k.w, own * x.w);
    }
  }
  store_four(query ? (T*)a.q_out + ((size_t)t * a.heads + h) * dim + d
             : value ? base + value_at(a.cache, page, h, at) + d : base + key_at(a.cache, page, h, at) + d, x);
}

template <typename T>
int launch_fours(const PrepareArgs& a, int units, cudaStream_t stream) {
  const int longest = a.cache.key_dim > a.cache.value_dim ? a.cache.key_dim : a.cache.value_dim;
  auto go = [&](auto kernel, int lanes) {
    const int per_block = WARPS * 32 / lanes;
    return dllm_launch_pdl(kernel, dim3(a.tokens, (units + per_block - 1) / per_block), dim3(WARPS * 32), 0, stream, a);
  };
  if (longest <= 32) return go(qkv_prepare_fours_kernel<T, 8>, 8);
  if (longest <= 64) return go(qkv_prepare_fours_kernel<T, 16>, 16);
  return go(qkv_prepare_fours_kernel<T, 32>, 32);
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
  const uintptr_t addresses = (uintptr_t)rows | (uintptr_t)q_bias | (uintptr_t)k_bias | (uintptr_t)v_bias |
                              (uintptr_t)q_weight | (uintptr_t)k_weight | (uintptr_t)table | (uintptr_t)first |
                              (uintptr_t)q_out | (uintptr_t)cache_base;
  if (((dim | vdim | q_at | k_at | v_at | stride) & 3) == 0 && (rotary_dim & 7) == 0 && dim <= 128 && vdim <= 128 &&
      (addresses & 15) == 0) {
    if (dtype == DLLM_F32) return launch_fours<float>(a, units, stream);
    if (dtype == DLLM_BF16) return launch_fours<__nv_bfloat16>(a, units, stream);
  }
  dim3 grid(tokens, (units + WARPS - 1) / WARPS), block(WARPS * 32);
  if (dtype == DLLM_F32) return dllm_launch_pdl(qkv_prepare_kernel<float>, grid, block, 0, stream, a);
  if (dtype == DLLM_BF16) return dllm_launch_pdl(qkv_prepare_kernel<__nv_bfloat16>, grid, block, 0, stream, a);
  return DLLM_BAD_ARGUMENT;
}
