// What happens to the residual stream behind a sublayer whose output is normed, as one kernel per row of the stream:
//
//   v = x + y / sqrt(mean(y^2) + eps) * w                     the output's norm and the residual sum
//   kept_before <- x, kept_after <- v                         (optional: results that later layers' sums read)
//   x <- v, or x <- sum_(j < terms) c_j X_j + c_terms v       the weighted sum over earlier layers' results
//   normed <- x / sqrt(mean(x^2) + next_eps) * next_w         (optional: the next product's operand, rounded once)
//
// Everything is float32 up to the operand. A row is a block's work, held in registers; where the step has few rows a
// cluster of two, four or eight blocks shares a row (each takes a run of its columns, the two sums of squares meet
// through distributed shared memory), since reading many earlier results by one multiprocessor would take as long as
// a product. A row's sums are formed in an order that depends only on the launch's shape.
#include "common.cuh"

namespace {
struct UpdateArgs {
  float* x;
  const float* y;
  const float* w;
  float eps;
  float* kept_before;     // [rows, hidden] or null
  float* kept_after;      // [rows, hidden] or null
  const float* earlier;   // X_j at earlier + j * stride
  long long stride;
  int terms;              // earlier results in the sum (c has terms + 1 values)
  const float* c;         // null: no sum
  int first_is_x;         // X_0 is this row of x as it was (kept_before has just been given it)
  const float* next_w;    // null: no norm
  float next_eps;
  void* normed;
  int hidden, cluster;
};

__device__ __forceinline__ float remote_value(const float* local, unsigned rank) {
  unsigned address = (unsigned)__cvta_generic_to_shared(local), remote;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(address), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
  return v;
}
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n"
               "barrier.cluster.wait.acquire.aligned;\n" ::: "memory");
}

// The sum over the row: over the block's threads, then over the cluster's blocks in rank order. `scratch` [33] floats
// of shared memory used by this call alone.
__device__ __forceinline__ float row_sum(float v, float* scratch, int cluster) {
  int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  v = warp_sum(v);
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float total = 0.f;
  for (int i = 0; i < warps; ++i) total += scratch[i];
  if (cluster == 1) return total;
  if (threadIdx.x == 0) scratch[32] = total;
  cluster_sync();
  total = 0.f;
  for (int r = 0; r < cluster; ++r) total += remote_value(scratch + 32, r);
  return total;
}

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<unsigned*>(&lo), *reinterpret_cast<unsigned*>(&hi));
}

template <typename T, int VPT>
__global__ void __launch_bounds__(256) stream_update_kernel(UpdateArgs a) {
  __shared__ float scratch[2][33];
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x / a.cluster, rank = blockIdx.x - row * a.cluster;
  const int pieces = a.hidden >> 2, per = (pieces + a.cluster - 1) / a.cluster;
  const int begin = rank * per, end = min(pieces, begin + per);
  const size_t base = (size_t)row * a.hidden;
  float4 x[VPT], y[VPT], sum[VPT];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    int p = begin + threadIdx.x + i * blockDim.x;
    x[i] = y[i] = sum[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (p < end) {
      y[i] = *reinterpret_cast<const float4*>(a.y + base + 4 * p);
      x[i] = *reinterpret_cast<const float4*>(a.x + base + 4 * p);
    }
  }
  if (a.c != nullptr) {
    int j = 0;
    if (a.first_is_x) {
      float c = a.c[0];
#pragma unroll
      for (int i = 0; i < VPT; ++i) sum[i] = make_float4(c * x[i].x, c * x[i].y, c * x[i].z, c * x[i].w);
      j = 1;
    }
#pragma unroll 4
    for (; j < a.terms; ++j) {
      float c = a.c[j];
      const float* from = a.earlier + (size_t)j * a.stride + base;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        int p = begin + threadIdx.x + i * blockDim.x;
        if (p < end) {
          float4 v = *reinterpret_cast<const float4*>(from + 4 * p);
          sum[i].x = fmaf(c, v.x, sum[i].x); sum[i].y = fmaf(c, v.y, sum[i].y);
          sum[i].z = fmaf(c, v.z, sum[i].z); sum[i].w = fmaf(c, v.w, sum[i].w);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    ss = fmaf(y[i].x, y[i].x, ss); ss = fmaf(y[i].y, y[i].y, ss);
    ss = fmaf(y[i].z, y[i].z, ss); ss = fmaf(y[i].w, y[i].w, ss);
  }
  float inv = 1.0f / sqrtf(row_sum(ss, scratch[0], a.cluster) / (float)a.hidden + a.eps);
  float last = a.c != nullptr ? a.c[a.terms] : 1.f;
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    int p = begin + threadIdx.x + i * blockDim.x;
    if (p >= end) continue;
    float4 w = *reinterpret_cast<const float4*>(a.w + 4 * p);
    if (a.kept_before != nullptr) store4(a.kept_before + base + 4 * p, x[i]);
    float4 v = make_float4(fmaf(y[i].x * inv, w.x, x[i].x), fmaf(y[i].y * inv, w.y, x[i].y),
                           fmaf(y[i].z * inv, w.z, x[i].z), fmaf(y[i].w * inv, w.w, x[i].w));
    if (a.kept_after != nullptr) store4(a.kept_after + base + 4 * p, v);
    if (a.c != nullptr)
      v = make_float4(fmaf(last, v.x, sum[i].x), fmaf(last, v.y, sum[i].y), fmaf(last, v.z, sum[i].z),
                      fmaf(last, v.w, sum[i].w));
    store4(a.x + base + 4 * p, v);
    x[i] = v;
    ss = fmaf(v.x, v.x, ss); ss = fmaf(v.y, v.y, ss); ss = fmaf(v.z, v.z, ss); ss = fmaf(v.w, v.w, ss);
  }
  if (a.next_w != nullptr) {
    float next = 1.0f / sqrtf(row_sum(ss, scratch[1], a.cluster) / (float)a.hidden + a.next_eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      int p = begin + threadIdx.x + i * blockDim.x;
      if (p >= end) continue;
      float4 w = *reinterpret_cast<const float4*>(a.next_w + 4 * p);
      store4((T*)a.normed + base + 4 * p, make_float4(x[i].x * next * w.x, x[i].y * next * w.y, x[i].z * next * w.z,
                                                      x[i].w * next * w.w));
    }
  }
  if (a.cluster > 1) cluster_sync();  // nobody leaves while another block may still read its sums
}

template <typename T, int VPT>
int launch(const UpdateArgs& a, int rows, int threads, cudaStream_t stream) {
  cudaLaunchConfig_t config = {};
  config.gridDim = dim3((unsigned)(rows * a.cluster));
  config.blockDim = dim3(threads);
  config.stream = stream;
  cudaLaunchAttribute attributes[2];
  int count = 0;
  if (a.cluster > 1) {
    attributes[count].id = cudaLaunchAttributeClusterDimension;
    attributes[count].val.clusterDim.x = a.cluster;
    attributes[count].val.clusterDim.y = 1;
    attributes[count].val.clusterDim.z = 1;
    ++count;
  }
  if (dllm_pdl_enabled()) {
    attributes[count].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[count].val.programmaticStreamSerializationAllowed = 1;
    ++count;
  }
  config.attrs = attributes;
  config.numAttrs = count;
  return cudaLaunchKernelEx(&config, stream_update_kernel<T, VPT>, a) == cudaSuccess ? DLLM_OK : DLLM_LAUNCH_FAILED;
}

template <typename T>
int launch_rows(UpdateArgs& a, int rows, cudaStream_t stream) {
  int pieces = a.hidden >> 2;
  a.cluster = 1;
  while (a.cluster < 8 && (long long)rows * a.cluster * 2 <= 148 && pieces / (a.cluster * 2) >= 32) a.cluster *= 2;
  int per = (pieces + a.cluster - 1) / a.cluster;
  int threads = per >= 256 ? 256 : ((per + 31) / 32) * 32;
  int each = (per + threads - 1) / threads;
  if (each <= 1) return launch<T, 1>(a, rows, threads, stream);
  if (each <= 2) return launch<T, 2>(a, rows, threads, stream);
  if (each <= 4) return launch<T, 4>(a, rows, threads, stream);
  if (each <= 8) return launch<T, 8>(a, rows, threads, stream);
  return DLLM_UNSUPPORTED_SIZE;
}
}  // namespace

// x, y [rows, hidden] float32, w [hidden]; see the top of the file. `earlier` + j * stride: the j-th earlier result
// (j < terms; j = 0 is read from x itself with first_is_x), c: terms + 1 coefficients on the device, or null for no sum.
// hidden: a multiple of 4 up to 8192.
DLLM_EXPORT int dllm_stream_update(float* x, const float* y, const float* w, float eps, float* kept_before,
                                   float* kept_after, const float* earlier, long long stride, int terms, const float* c,
                                   int first_is_x, const float* next_w, float next_eps, void* normed, int rows,
                                   int hidden, int dtype, cudaStream_t stream) {
  if (rows <= 0) return DLLM_OK;
  if (hidden <= 0 || (hidden & 3) || hidden > 8192) return DLLM_UNSUPPORTED_SIZE;
  if (!x || !y || !w || (next_w != nullptr && normed == nullptr) || terms < 0 ||
      (c != nullptr && terms > (first_is_x ? 1 : 0) && earlier == nullptr))
    return DLLM_BAD_ARGUMENT;
  UpdateArgs a = {x, y, w, eps, kept_before, kept_after, earlier, stride, terms, c, first_is_x, next_w, next_eps, normed,
                  hidden, 1};
  if (dtype == DLLM_F32) return launch_rows<float>(a, rows, stream);
  if (dtype == DLLM_BF16) return launch_rows<__nv_bfloat16>(a, rows, stream);
  return DLLM_BAD_ARGUMENT;
}
