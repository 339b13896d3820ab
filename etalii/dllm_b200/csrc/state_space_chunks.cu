// State-space duality over prompts as products of small matrices: the recurrence of recurrent.cu,
//
//   S_t = a_t S_(t-1) + b_t B_t x_t^T,   y_t = S_t^T C_t + skip x_t,
//
// in chunks of 64 tokens. With l_t the sum of the logarithms of a over the chunk up to t and S the state in front of it,
//
//   y_t = e^(l_t) S^T C_t + sum_(s <= t) e^(l_t - l_s) b_s (C_t . B_s) x_s + skip x_t,
//
// and the chunk leaves e^(l_last) S + sum_s e^(l_last - l_s) b_s B_s x_s^T. Three kernels:
//
//   left:    per chunk, head and 64 columns: what the chunk leaves of a zero state (a product over its tokens);
//   starts:  per head and element, chunk after chunk: from that what every chunk starts from, and the final state;
//   chunks:  per chunk, head and 64 columns: y, with the products C S, C B^T and (weighted C B^T) x.
//
// The products run on the tensor cores (mma.sync m16n8k16 bfloat16) with every float32 operand as the sum of two bfloat16
// values, v = hi + lo, and hi hi + hi lo + lo hi summed in float32: a product's relative error is about 2^-16, where one
// bfloat16 value would leave 2^-9. Logarithms are summed in float64 and only their differences, which are never
// positive, go through the exponential. States and sums are float32.
//
// State layout: [slot][head][column][row], as the scan's.
#include "common.cuh"

namespace {
typedef __nv_bfloat16 bf16;
// (a block's warps: four times sixteen rows of a tile, two halves of its columns)
constexpr int CHUNK = 64, COLS = 64, WARPS = 8, THREADS = WARPS * 32;
constexpr int LDX = COLS + 8;

struct ChunkArgs {
  const float* prepared;  // a token's x (heads * vdim) | B (groups * dim) | C (groups * dim), rows of `stride` floats
  int stride;
  const float* aux;       // a token's step size b of head h at aux[token * aux_stride + heads + h]
  int aux_stride;
  const float* a_log;     // [heads]: log a = -exp(a_log) b
  const float* skip;      // [heads]
  int heads, groups, dim, vdim;
  float* state;           // [slots][heads][vdim][dim]
  float* starts;          // [sequences * chunks][heads][vdim][dim]: what a chunk leaves, then what it starts from
  float* decays;          // [sequences * chunks][heads]: e^(l_last)
  const int* cu_seqlens;
  const int* slots;
  int chunks;             // the most chunks a sequence has
  float* out;             // [tokens][heads * vdim]
};

__device__ __forceinline__ void ldmatrix_x4(unsigned* r, const void* p) {
  unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned* r, const void* p) {
  unsigned s = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float* c, const unsigned* a, unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two columns of eight of the right operand: both parts of both operands, but lo lo.
__device__ __forceinline__ void mma_split(float* c0, float* c1, const unsigned* a_hi, const unsigned* a_lo,
                                          const unsigned* b_hi, const unsigned* b_lo) {
  mma_bf16(c0, a_lo, b_hi[0], b_hi[1]);
  mma_bf16(c1, a_lo, b_hi[2], b_hi[3]);
  mma_bf16(c0, a_hi, b_lo[0], b_lo[1]);
  mma_bf16(c1, a_hi, b_lo[2], b_lo[3]);
  mma_bf16(c0, a_hi, b_hi[0], b_hi[1]);
  mma_bf16(c1, a_hi, b_hi[2], b_hi[3]);
}
// Two values as hi and lo parts.
__device__ __forceinline__ void split2(float x, float y, unsigned& hi, unsigned& lo) {
  __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  float2 back = __bfloat1622float2(h);
  __nv_bfloat162 l = __floats2bfloat162_rn(x - back.x, y - back.y);
  hi = *reinterpret_cast<unsigned*>(&h);
  lo = *reinterpret_cast<unsigned*>(&l);
}

// A tile of 64 rows x PAD values on its way from global memory: asked for (`rows` rows of `cols` values, zeros elsewhere),
// then put into hi and lo tiles [64][PAD + 8]; row r times factor[r] if given.
template <int PAD>
struct Tile {
  static constexpr int FOURS = PAD / 4, LD = PAD + 8, PIECES = 64 * FOURS / THREADS;
  float4 v[PIECES];
  __device__ __forceinline__ void ask(const float* src, size_t stride, int rows, int cols) {
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
      const int i = threadIdx.x + p * THREADS, r = i / FOURS, c = 4 * (i % FOURS);
      v[p] = r < rows && c < cols ? *reinterpret_cast<const float4*>(src + (size_t)r * stride + c)
                                  : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  __device__ __forceinline__ void put(bf16* hi, bf16* lo, const float* factor = nullptr) {
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
      const int i = threadIdx.x + p * THREADS, r = i / FOURS, c = 4 * (i % FOURS);
      float4 x = v[p];
      if (factor != nullptr) {
        const float f = factor[r];
        x.x *= f; x.y *= f; x.z *= f; x.w *= f;
      }
      uint2 h, l;
      split2(x.x, x.y, h.x, l.x);
      split2(x.z, x.w, h.y, l.y);
      *reinterpret_cast<uint2*>(hi + r * LD + c) = h;
      *reinterpret_cast<uint2*>(lo + r * LD + c) = l;
    }
  }
};

// The chunk's tokens: how many, the first one's row; their step sizes, and the running sums of log a (beyond the last
// token the step size is zero and the sum stays).
struct Chunk {
  int seq, part, first, count;
  __device__ __forceinline__ Chunk(const ChunkArgs& a) {
    seq = blockIdx.z / a.chunks;
    part = blockIdx.z % a.chunks;
    first = a.cu_seqlens[seq] + part * CHUNK;
    count = min(CHUNK, a.cu_seqlens[seq + 1] - first);
  }
};
__device__ __forceinline__ void sum_logs(const ChunkArgs& a, const Chunk& chunk, int head, double* sums, float* steps) {
  if (threadIdx.x < 32) {  // lane i: the tokens 2 i and 2 i + 1
    const double rate = -(double)expf(a.a_log[head]);
    float b[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int t = 2 * threadIdx.x + j;
      b[j] = t < chunk.count ? a.aux[(size_t)(chunk.first + t) * a.aux_stride + a.heads + head] : 0.f;
      steps[t] = b[j];
    }
    const double l0 = rate * b[0], pair = l0 + rate * b[1];
    double upto = pair;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      double before = __shfl_up_sync(0xffffffffu, upto, o);
      if ((int)threadIdx.x >= o) upto += before;
    }
    sums[2 * threadIdx.x] = upto - pair + l0;
    sums[2 * threadIdx.x + 1] = upto;
  }
}

template <int N>
__global__ void __launch_bounds__(THREADS) left_kernel(ChunkArgs a) {
  constexpr int LDN = N + 8;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* b_hi = reinterpret_cast<bf16*>(smem);  // [64][LDN] tokens x rows of S
  bf16* b_lo = b_hi + 64 * LDN;
  bf16* x_hi = b_lo + 64 * LDN;                // [64][LDX] tokens x columns, weighted
  bf16* x_lo = x_hi + 64 * LDX;
  __shared__ double sums[CHUNK];
  __shared__ float steps[CHUNK], factor[CHUNK];
  pdl_launch_dependents();
  pdl_wait();
  const Chunk chunk(a);
  if (chunk.count <= 0) return;
  const int head = blockIdx.y, col0 = blockIdx.x * COLS, group = head / (a.heads / a.groups);
  const int inner = a.heads * a.vdim, cols = min(COLS, a.vdim - col0);
  const float* row = a.prepared + (size_t)chunk.first * a.stride;
  Tile<N> b;
  Tile<COLS> x;
  b.ask(row + inner + group * a.dim, a.stride, chunk.count, a.dim);
  x.ask(row + head * a.vdim + col0, a.stride, chunk.count, cols);
  sum_logs(a, chunk, head, sums, steps);
  b.put(b_hi, b_lo);
  __syncthreads();
  if (threadIdx.x < CHUNK) factor[threadIdx.x] = steps[threadIdx.x] * expf((float)(sums[CHUNK - 1] - sums[threadIdx.x]));
  __syncthreads();
  x.put(x_hi, x_lo, factor);
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, mat = lane >> 3, n0 = (threadIdx.x >> 7) * (N / 2);
  float acc[N / 16][4];
#pragma unroll
  for (int i = 0; i < N / 16; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll
  for (int k = 0; k < CHUNK / 16; ++k) {
    unsigned xh[4], xl[4];  // the warp's sixteen columns as rows, sixteen tokens
    const int at = (k * 16 + (mat >> 1) * 8 + (lane & 7)) * LDX + warp * 16 + (mat & 1) * 8;
    ldmatrix_x4_trans(xh, x_hi + at);
    ldmatrix_x4_trans(xl, x_lo + at);
#pragma unroll
    for (int n = 0; n < N / 32; ++n) {
      unsigned bh[4], bl[4];
      const int from = (k * 16 + (mat & 1) * 8 + (lane & 7)) * LDN + n0 + n * 16 + (mat >> 1) * 8;
      ldmatrix_x4_trans(bh, b_hi + from);
      ldmatrix_x4_trans(bl, b_lo + from);
      mma_split(acc[2 * n], acc[2 * n + 1], xh, xl, bh, bl);
    }
  }
  float* dst = a.starts + ((size_t)blockIdx.z * a.heads + head) * a.vdim * a.dim;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int col = col0 + warp * 16 + (lane >> 2) + 8 * half;
    if (col >= a.vdim) continue;
#pragma unroll
    for (int i = 0; i < N / 16; ++i) {
      const int n = n0 + i * 8 + (lane & 3) * 2;
      if (n < a.dim)
        *reinterpret_cast<float2*>(dst + (size_t)col * a.dim + n) = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
    }
  }
  if (blockIdx.x == 0 && threadIdx.x == 0) a.decays[(size_t)blockIdx.z * a.heads + head] = expf((float)sums[CHUNK - 1]);
}

// A thread per four elements of a head's matrix; the chunks' loads are asked for several ahead of the state that walks
// through them.
__global__ void __launch_bounds__(128) starts_kernel(ChunkArgs a) {
  constexpr int AHEAD = 6;
  pdl_launch_dependents();
  pdl_wait();
  const int head = blockIdx.y, seq = blockIdx.z;
  const int fours = a.vdim * a.dim / 4, i = blockIdx.x * blockDim.x + threadIdx.x;
  const int parts = (a.cu_seqlens[seq + 1] - a.cu_seqlens[seq] + CHUNK - 1) / CHUNK;
  if (i >= fours || parts <= 0) return;
  float4* whole = reinterpret_cast<float4*>(a.state + ((size_t)a.slots[seq] * a.heads + head) * a.vdim * a.dim) + i;
  const size_t first = (size_t)seq * a.chunks * a.heads + head;
  float4* kept = reinterpret_cast<float4*>(a.starts + first * a.vdim * a.dim) + i;
  const size_t step = (size_t)a.heads * fours;
  const float* decays = a.decays + first;
  float4 s = *whole, left[2][AHEAD];
  float decay[2][AHEAD];
  auto ask = [&](int p0, int buffer) {
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (p0 + j < parts) {
        left[buffer][j] = kept[(p0 + j) * step];
        decay[buffer][j] = decays[(size_t)(p0 + j) * a.heads];
      }
  };
  auto walk = [&](int p0, int buffer) {
#pragma unroll
    for (int j = 0; j < AHEAD; ++j)
      if (p0 + j < parts) {
        kept[(p0 + j) * step] = s;
        const float4 l = left[buffer][j];
        const float d = decay[buffer][j];
        s.x = fmaf(d, s.x, l.x); s.y = fmaf(d, s.y, l.y); s.z = fmaf(d, s.z, l.z); s.w = fmaf(d, s.w, l.w);
      }
  };
  ask(0, 0);
  for (int p0 = 0; p0 < parts; p0 += 2 * AHEAD) {
    ask(p0 + AHEAD, 1);
    walk(p0, 0);
    ask(p0 + 2 * AHEAD, 0);
    walk(p0 + AHEAD, 1);
  }
  *whole = s;
}

template <int N>
__global__ void __launch_bounds__(THREADS) chunks_kernel(ChunkArgs a) {
  constexpr int LDN = N + 8;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* c_hi = reinterpret_cast<bf16*>(smem);  // [64][LDN] tokens x rows of S
  bf16* c_lo = c_hi + 64 * LDN;
  bf16* b_hi = c_lo + 64 * LDN;                // first S (columns x rows), then B (tokens x rows)
  bf16* b_lo = b_hi + 64 * LDN;
  bf16* x_hi = b_lo + 64 * LDN;                // [64][LDX] tokens x columns
  bf16* x_lo = x_hi + 64 * LDX;
  __shared__ double sums[CHUNK];
  __shared__ float steps[CHUNK];
  pdl_launch_dependents();
  pdl_wait();
  const Chunk chunk(a);
  if (chunk.count <= 0) return;
  const int head = blockIdx.y, col0 = blockIdx.x * COLS, group = head / (a.heads / a.groups);
  const int inner = a.heads * a.vdim, cols = min(COLS, a.vdim - col0);
  const float* row = a.prepared + (size_t)chunk.first * a.stride;
  const float* x = row + head * a.vdim + col0;
  Tile<N> b;
  {
    Tile<N> c;
    Tile<COLS> xs;
    c.ask(row + inner + (a.groups + group) * a.dim, a.stride, chunk.count, a.dim);
    b.ask(a.starts + (((size_t)blockIdx.z * a.heads + head) * a.vdim + col0) * a.dim, a.dim, cols, a.dim);
    xs.ask(x, a.stride, chunk.count, cols);
    sum_logs(a, chunk, head, sums, steps);
    c.put(c_hi, c_lo);
    b.put(b_hi, b_lo);
    xs.put(x_hi, x_lo);
  }
  b.ask(row + inner + group * a.dim, a.stride, chunk.count, a.dim);  // (on its way while the products with S run)
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = (threadIdx.x >> 5) & 3, mat = lane >> 3, g = lane >> 2, t = lane & 3;
  const int v0 = (threadIdx.x >> 7) * (COLS / 2);  // the warp's columns
  const int c_at = (warp * 16 + (lane & 15)) * LDN + (lane >> 4) * 8;       // the left operand's sixteen tokens
  const int b_at = ((mat >> 1) * 8 + (lane & 7)) * LDN + (mat & 1) * 8;     // sixteen rows of a right operand
  float acc[COLS / 16][4];
#pragma unroll
  for (int i = 0; i < COLS / 16; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // what the state in front of the chunk answers
#pragma unroll
  for (int k = 0; k < N / 16; ++k) {
    unsigned ch[4], cl[4];
    ldmatrix_x4(ch, c_hi + c_at + k * 16);
    ldmatrix_x4(cl, c_lo + c_at + k * 16);
#pragma unroll
    for (int n = 0; n < COLS / 32; ++n) {
      unsigned sh[4], sl[4];
      ldmatrix_x4(sh, b_hi + b_at + (v0 + n * 16) * LDN + k * 16);
      ldmatrix_x4(sl, b_lo + b_at + (v0 + n * 16) * LDN + k * 16);
      mma_split(acc[2 * n], acc[2 * n + 1], ch, cl, sh, sl);
    }
  }
  const double own[2] = {sums[warp * 16 + g], sums[warp * 16 + g + 8]};  // this thread's two tokens
  const float reach[2] = {expf((float)own[0]), expf((float)own[1])};
#pragma unroll
  for (int i = 0; i < COLS / 16; ++i) {
    acc[i][0] *= reach[0]; acc[i][1] *= reach[0];
    acc[i][2] *= reach[1]; acc[i][3] *= reach[1];
  }
  __syncthreads();  // S has been read by all
  b.put(b_hi, b_lo);
  __syncthreads();
  // the chunk's own tokens, sixteen at a time and none behind the warp's last
#pragma unroll
  for (int j = 0; j < CHUNK / 16; ++j) {
    if (j > warp) break;
    float s[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int r = 0; r < 4; ++r) s[i][r] = 0.f;
#pragma unroll
    for (int k = 0; k < N / 16; ++k) {
      unsigned ch[4], cl[4], bh[4], bl[4];
      ldmatrix_x4(ch, c_hi + c_at + k * 16);
      ldmatrix_x4(cl, c_lo + c_at + k * 16);
      ldmatrix_x4(bh, b_hi + b_at + j * 16 * LDN + k * 16);
      ldmatrix_x4(bl, b_lo + b_at + j * 16 * LDN + k * 16);
      mma_split(s[0], s[1], ch, cl, bh, bl);
    }
    unsigned ph[4], pl[4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float p[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int from = j * 16 + i * 8 + t * 2 + r;
          p[r] = from <= warp * 16 + g + 8 * half
                     ? s[i][2 * half + r] * steps[from] * expf((float)(own[half] - sums[from])) : 0.f;
        }
        split2(p[0], p[1], ph[2 * i + half], pl[2 * i + half]);
      }
#pragma unroll
    for (int n = 0; n < COLS / 32; ++n) {
      unsigned xh[4], xl[4];
      const int at = (j * 16 + (mat & 1) * 8 + (lane & 7)) * LDX + v0 + n * 16 + (mat >> 1) * 8;
      ldmatrix_x4_trans(xh, x_hi + at);
      ldmatrix_x4_trans(xl, x_lo + at);
      mma_split(acc[2 * n], acc[2 * n + 1], ph, pl, xh, xl);
    }
  }
  const float share = a.skip[head];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int token = warp * 16 + g + 8 * half;
    if (token >= chunk.count) continue;
    float* dst = a.out + (size_t)(chunk.first + token) * inner + head * a.vdim + col0;
    const float* own_x = x + (size_t)token * a.stride;
#pragma unroll
    for (int i = 0; i < COLS / 16; ++i) {
      const int c = v0 + i * 8 + t * 2;
      if (c >= cols) continue;
      const float2 xv = *reinterpret_cast<const float2*>(own_x + c);
      *reinterpret_cast<float2*>(dst + c) = make_float2(fmaf(share, xv.x, acc[i][2 * half]),
                                                        fmaf(share, xv.y, acc[i][2 * half + 1]));
    }
  }
}

template <int N>
int launch(const ChunkArgs& a, int sequences, cudaStream_t stream) {
  constexpr size_t left_bytes = (size_t)2 * 64 * (N + 8 + LDX) * sizeof(bf16);
  constexpr size_t chunk_bytes = (size_t)2 * 64 * (2 * (N + 8) + LDX) * sizeof(bf16);
  static bool allowed = false;
  if (!allowed) {
    if (cudaFuncSetAttribute(left_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)left_bytes) != cudaSuccess ||
        cudaFuncSetAttribute(chunks_kernel<N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)chunk_bytes) != cudaSuccess)
      return DLLM_LAUNCH_FAILED;
    allowed = true;
  }
  const dim3 grid((a.vdim + COLS - 1) / COLS, a.heads, sequences * a.chunks);
  int status = dllm_launch_pdl(left_kernel<N>, grid, dim3(THREADS), left_bytes, stream, a);
  if (status != DLLM_OK) return status;
  status = dllm_launch_pdl(starts_kernel, dim3((a.vdim * a.dim / 4 + 127) / 128, a.heads, sequences), dim3(128), 0, stream,
                           a);
  if (status != DLLM_OK) return status;
  return dllm_launch_pdl(chunks_kernel<N>, grid, dim3(THREADS), chunk_bytes, stream, a);
}
}  // namespace

// prepared [tokens][stride] = [x | B | C] and aux as `dllm_state_space_prepare` leaves them; `longest`: the most new tokens a
// sequence of the step has; starts and decays: scratch for ceil(longest / 64) chunks a sequence (see ChunkArgs). dim a
// multiple of 4 up to 128, vdim of 4; everything 16-byte aligned.
DLLM_EXPORT int dllm_state_space_chunks(const float* prepared, int stride, const float* aux, int aux_stride,
                                        const float* a_log, const float* skip, int heads, int groups, int dim, int vdim,
                                        float* state, float* starts, float* decays, const int* cu_seqlens,
                                        const int* slots, int sequences, int longest, float* out, cudaStream_t stream) {
  if (sequences <= 0 || longest <= 0) return DLLM_OK;
  const int chunks = (longest + CHUNK - 1) / CHUNK;
  if (heads <= 0 || heads > 65535 || groups <= 0 || heads % groups || dim <= 0 || dim > 128 || (dim & 3) || vdim <= 0 ||
      (vdim & 3) || (stride & 3) || stride < heads * vdim + 2 * groups * dim || aux_stride < 2 * heads ||
      (long long)sequences * chunks > 65535)
    return DLLM_UNSUPPORTED_SIZE;
  if (!prepared || !aux || !a_log || !skip || !state || !starts || !decays || !cu_seqlens || !slots || !out ||
      (((uintptr_t)prepared | (uintptr_t)state | (uintptr_t)starts | (uintptr_t)out) & 15))
    return DLLM_BAD_ARGUMENT;
  const ChunkArgs a = {prepared, stride, aux, aux_stride, a_log, skip, heads, groups, dim, vdim, state, starts, decays,
                       cu_seqlens, slots, chunks, out};
  if (dim <= 32) return launch<32>(a, sequences, stream);
  if (dim <= 64) return launch<64>(a, sequences, stream);
  return launch<128>(a, sequences, stream);
}
