// The experts' products of a prompt-sized step on the 5th-generation tensor cores (bfloat16, float32 accumulation in tensor
// memory). The (token, choice) pairs are in expert order (moe_grouped.cu: `moe_sort`), and so are the rows of the left
// operand: `moe_gather` copies the tokens' activations there for the first product, whose results are in that order for
// the second. A persistent block takes tiles of 128 places of ONE expert x 256 output features; which tiles there are it
// finds from the experts' offsets on the device, so a step's launches do not depend on what the router chose.
//
//   warp 0     one lane issues TMA loads of 128 x 64 places and 256 x 64 rows of the expert's matrix (the stacked matrices
//              are one of experts x n rows) into a ring of four stages; rows of other experts that a tile's edge brings
//              along give results that are never stored;
//   warp 1     tensor memory; one lane issues tcgen05.mma, two accumulators in turn;
//   warps 2-9  the epilogue of one tile under the products of the next: an activation or gated unit and a bfloat16 row in
//              expert order, or the float32 row scattered to its pair.
//
// Every wait is bounded: a role that gives up records a status word and leaves, the block still frees its tensor memory.
#include "expert_unit.cuh"
#include "tcgen05.cuh"

namespace {
using namespace tc5;
typedef __nv_bfloat16 bf16;
constexpr int BM = 128, BN = 256, BK = 64, STAGES = 4, MAX_EXPERTS = 256;
constexpr int EPI_WARPS = 8, THREADS = 64 + 32 * EPI_WARPS;
constexpr int A_BYTES = BM * BK * 2, B_BYTES = BN * BK * 2;
constexpr size_t SMEM = (size_t)STAGES * (A_BYTES + B_BYTES) + 1024;
constexpr int EPI_GLU = 0, EPI_SCATTER = 1, EPI_ACT = 2;

struct GroupedArgs {
  int n, k, experts;
  const int* offsets;     // [experts + 1]: where each expert's places begin
  const int* place_pair;  // place -> pair
  bf16* act;              // EPI_GLU: [places, n / 2]; EPI_ACT: [places, n]
  float* y;               // EPI_SCATTER: [pairs, n]
  float limit, alpha, shift;
  int kind;
};

template <int EPI>
__global__ void __launch_bounds__(THREADS, 1) grouped_tcgen05_kernel(const __grid_constant__ CUtensorMap map_a,
                                                                     const __grid_constant__ CUtensorMap map_w,
                                                                     GroupedArgs g, int* __restrict__ status) {
  extern __shared__ unsigned char smem_raw[];
  unsigned char* tiles = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);  // swizzle atoms: 1 KB
  __shared__ uint64_t full_bar[STAGES], empty_bar[STAGES], acc_full[2], acc_empty[2];
  __shared__ unsigned tmem_base_s;
  __shared__ int offsets[MAX_EXPERTS + 1], first_tile[MAX_EXPERTS + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&acc_full[i], 1); mbar_init(&acc_empty[i], EPI_WARPS); }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) tmem_alloc(&tmem_base_s, 2 * BN);
  pdl_wait();
  for (int e = threadIdx.x; e <= g.experts; e += THREADS) offsets[e] = g.offsets[e];
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const unsigned tmem_base = tmem_base_s;
  if (warp == 0) {  // how many tiles the experts before each one have
    int before = 0;
    for (int e0 = 0; e0 < g.experts; e0 += 32) {
      const int e = e0 + lane, mine = e < g.experts ? (offsets[e + 1] - offsets[e] + BM - 1) / BM : 0;
      int upto = mine;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        int left = __shfl_up_sync(0xffffffffu, upto, o);
        if (lane >= o) upto += left;
      }
      if (e < g.experts) first_tile[e] = before + upto - mine;
      before += __shfl_sync(0xffffffffu, upto, 31);
    }
    if (lane == 0) first_tile[g.experts] = before;
  }
  __syncthreads();
  const int m_tiles = first_tile[g.experts], items = m_tiles * ((g.n + BN - 1) / BN), k_tiles = (g.k + BK - 1) / BK;
  struct Tile { int expert, m0, rows, n0; };
  auto tile_of = [&](int item) {
    const int m = item % m_tiles;
    int lo = 0, hi = g.experts - 1;  // the last expert whose first tile is not behind m
    while (lo < hi) {
      int mid = (lo + hi + 1) >> 1;
      if (first_tile[mid] <= m) lo = mid; else hi = mid - 1;
    }
    Tile t;
    t.expert = lo;
    t.m0 = offsets[lo] + (m - first_tile[lo]) * BM;
    t.rows = min(BM, offsets[lo + 1] - t.m0);
    t.n0 = item / m_tiles * BN;
    return t;
  };

  if (warp == 0) {
    if (lane == 0) {
      asm volatile("prefetch.tensormap [%0];" ::"l"(&map_a) : "memory");
      asm volatile("prefetch.tensormap [%0];" ::"l"(&map_w) : "memory");
      int it = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < items && ok; item += gridDim.x) {
        const Tile t = tile_of(item);
        for (int kt = 0; kt < k_tiles; ++kt, ++it) {
          const int s = it % STAGES;
          if (it >= STAGES && !mbar_wait(&empty_bar[s], ((it / STAGES) - 1) & 1)) {
            *(volatile int*)status = 42;
            ok = false;
            break;
          }
          mbar_expect_tx(&full_bar[s], A_BYTES + B_BYTES);
          unsigned char* dst = tiles + (size_t)s * (A_BYTES + B_BYTES);
          tma_load_2d(dst, &map_a, &full_bar[s], kt * BK, t.m0);
          tma_load_2d(dst + A_BYTES, &map_w, &full_bar[s], kt * BK, t.expert * g.n + t.n0);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr unsigned idesc = instr_desc(BM, BN);
      int it = 0, lt = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < items && ok; item += gridDim.x, ++lt) {
        const int buf = lt & 1;
        if (lt >= 2 && !mbar_wait(&acc_empty[buf], ((lt >> 1) - 1) & 1)) { *(volatile int*)status = 45; break; }
        fence_after_sync();
        for (int kt = 0; kt < k_tiles; ++kt, ++it) {
          const int s = it % STAGES;
          if (!mbar_wait(&full_bar[s], (it / STAGES) & 1)) { *(volatile int*)status = 43; ok = false; break; }
          fence_after_sync();
          const unsigned a = smem_u32(tiles + (size_t)s * (A_BYTES + B_BYTES)), b = a + A_BYTES;
#pragma unroll
          for (int k = 0; k < BK / 16; ++k)
            umma(tmem_base + (unsigned)(buf * BN), smem_desc(a + k * 32), smem_desc(b + k * 32), idesc,
                 (kt > 0 || k > 0) ? 1u : 0u);
          tcgen05_commit(&empty_bar[s]);
        }
        tcgen05_commit(&acc_full[buf]);
      }
    }
  } else {
    const int quarter = warp & 3, c0 = ((warp - 2) >> 2) * (BN / 2);
    int lt = 0;
    for (int item = blockIdx.x; item < items; item += gridDim.x, ++lt) {
      const int buf = lt & 1, r = quarter * 32 + lane;
      const Tile t = tile_of(item);
      const bool exists = r < t.rows;
      const size_t place = t.m0 + r;
      const int pair = EPI == EPI_SCATTER && exists ? g.place_pair[place] : 0;
      if (!mbar_wait(&acc_full[buf], (lt >> 1) & 1)) {
        if (lane == 0) *(volatile int*)status = 44;
        break;
      }
      fence_after_sync();
      const unsigned acc = tmem_base + ((unsigned)(quarter * 32) << 16) + (unsigned)(buf * BN + c0);
#pragma unroll
      for (int c = 0; c < BN / 2; c += 16) {
        unsigned v[16];
        tmem_load16(acc + (unsigned)c, v);
        if (c + 16 == BN / 2) {  // this warp's last values are in registers: the accumulator may be reused
          fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&acc_empty[buf]);
        }
        const int n = t.n0 + c0 + c;
        float f[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) f[i] = __uint_as_float(v[i]);
        if (!exists || n >= g.n) {
        } else if (EPI == EPI_SCATTER) {
          float* dst = g.y + (size_t)pair * g.n + n;
#pragma unroll
          for (int i = 0; i < 16; i += 4)
            if (n + i + 4 <= g.n) *reinterpret_cast<float4*>(dst + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
        } else if (EPI == EPI_ACT) {
          bf16* dst = g.act + place * g.n + n;
#pragma unroll
          for (int i = 0; i < 16; i += 8) {
            uint4 o;
            __nv_bfloat162* po = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
            for (int j = 0; j < 4; ++j)
              po[j] = __floats2bfloat162_rn(plain_activation(f[i + 2 * j], g.kind),
                                            plain_activation(f[i + 2 * j + 1], g.kind));
            if (n + i + 8 <= g.n) *reinterpret_cast<uint4*>(dst + i) = o;
          }
        } else {  // (gate at even columns, up at odd ones; n is a multiple of 16)
          uint4 o;
          __nv_bfloat162* po = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
          for (int j = 0; j < 4; ++j)
            po[j] = __floats2bfloat162_rn(gated_unit(f[4 * j], f[4 * j + 1], g.limit, g.alpha, g.shift),
                                          gated_unit(f[4 * j + 2], f[4 * j + 3], g.limit, g.alpha, g.shift));
          *reinterpret_cast<uint4*>(g.act + place * (g.n / 2) + (n >> 1)) = o;
        }
        __syncwarp();  // (tensor memory is read by whole warps)
      }
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 2 * BN);
}

// rows[place] = h[place_pair[place] / top], 16 bytes a thread.
__global__ void __launch_bounds__(256) moe_gather_kernel(uint4* __restrict__ rows, const uint4* __restrict__ h,
                                                         const int* __restrict__ place_pair, int top, int pieces,
                                                         long long total) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long place = i / pieces;
    rows[i] = h[(long long)(place_pair[place] / top) * pieces + (i - place * pieces)];
  }
}

template <int EPI>
int launch(const void* a, const void* w, const GroupedArgs& g, int pairs, int* status, cudaStream_t stream) {
  if ((long long)g.experts * g.n > 0x7fffffffll) return DLLM_UNSUPPORTED_SIZE;
  if (status == nullptr || (((uintptr_t)a | (uintptr_t)w | (uintptr_t)g.act | (uintptr_t)g.y) & 15))
    return DLLM_BAD_ARGUMENT;
  alignas(64) CUtensorMap map_a, map_w;
  if (!make_map(&map_a, a, pairs, g.k, BM) || !make_map(&map_w, w, (long long)g.experts * g.n, g.k, BN))
    return DLLM_LAUNCH_FAILED;
  static int sms = 0;
  if (sms == 0) {
    int device = 0;
    if (cudaGetDevice(&device) != cudaSuccess ||
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device) != cudaSuccess || sms <= 0 ||
        cudaFuncSetAttribute(grouped_tcgen05_kernel<EPI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM) !=
            cudaSuccess) {
      sms = 0;
      return DLLM_LAUNCH_FAILED;
    }
  }
  // every expert's rows in tiles of BM: at most pairs / BM + experts of them
  const long long most = (long long)(pairs / BM + g.experts) * ((g.n + BN - 1) / BN);
  return dllm_launch_pdl(grouped_tcgen05_kernel<EPI>, dim3((unsigned)(most < sms ? most : sms)), dim3(THREADS), SMEM, stream,
                         map_a, map_w, g, status);
}

bool sizes_ok(int k, int n, int experts, int top) {
  return k > 0 && (k & 7) == 0 && n > 0 && (n & 7) == 0 && experts > 0 && experts <= MAX_EXPERTS && top > 0;
}
}  // namespace

// rows [pairs, width] bfloat16 in expert order from h [tokens, width]; width a multiple of 8.
DLLM_EXPORT int dllm_moe_gather(void* rows, const void* h, const int* place_pair, int width, int top, int pairs,
                                cudaStream_t stream) {
  if (pairs <= 0) return DLLM_OK;
  if (width <= 0 || (width & 7) || top <= 0) return DLLM_UNSUPPORTED_SIZE;
  if (!rows || !h || !place_pair || (((uintptr_t)rows | (uintptr_t)h) & 15)) return DLLM_BAD_ARGUMENT;
  const long long total = (long long)pairs * (width / 8);
  const int blocks = (int)((total + 255) / 256 < 148 * 16 ? (total + 255) / 256 : 148 * 16);
  return dllm_launch_pdl(moe_gather_kernel, dim3(blocks), dim3(256), 0, stream, (uint4*)rows, (const uint4*)h, place_pair,
                         top, width / 8, total);
}

// act [pairs, ff] bfloat16 in expert order from rows [pairs, width] in expert order: with kind 0 the gated unit of
// w_up [experts, 2 ff, width] (gate and up rows interleaved), else the activation `kind` of w_up [experts, ff, width].
DLLM_EXPORT int dllm_moe_grouped_tcgen05_up(void* act, const void* rows, int width, const void* w_up, int ff, int experts,
                                            int pairs, const int* offsets, int kind, float limit, float alpha, float shift,
                                            int* status, cudaStream_t stream) {
  if (pairs <= 0) return DLLM_OK;
  if (!sizes_ok(width, ff, experts, 1)) return DLLM_UNSUPPORTED_SIZE;
  if (!act || !rows || !w_up || !offsets || kind < 0 || kind > 3) return DLLM_BAD_ARGUMENT;
  const GroupedArgs g = {kind == 0 ? 2 * ff : ff, width, experts, offsets, nullptr, (bf16*)act, nullptr, limit, alpha, shift,
                         kind};
  return kind == 0 ? launch<EPI_GLU>(rows, w_up, g, pairs, status, stream)
                   : launch<EPI_ACT>(rows, w_up, g, pairs, status, stream);
}

// y [pairs, width] float32 by pair from act [pairs, ff] in expert order; w_down [experts, width, ff].
DLLM_EXPORT int dllm_moe_grouped_tcgen05_down(float* y, const void* act, int ff, const void* w_down, int width, int experts,
                                              int pairs, const int* offsets, const int* place_pair, int* status,
                                              cudaStream_t stream) {
  if (pairs <= 0) return DLLM_OK;
  if (!sizes_ok(ff, width, experts, 1)) return DLLM_UNSUPPORTED_SIZE;
  if (!y || !act || !w_down || !offsets || !place_pair) return DLLM_BAD_ARGUMENT;
  const GroupedArgs g = {width, ff, experts, offsets, place_pair, nullptr, y, 0.f, 0.f, 0.f, 0};
  return launch<EPI_SCATTER>(act, w_down, g, pairs, status, stream);
}
