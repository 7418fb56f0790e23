// Latent attention on a paged latent cache (bf16 or fp32).
//
// A token leaves one normalised latent c of `rank` values in the cache. With per-head matrices UK_n [dim, rank] and
// UV_n [vdim, rank], score = q_n . (UK_n c) = (UK_n^T q_n) . c and output = UV_n (sum_j p_j c_j): a decode step
// moves the two matrices to the query side and the output side, and every head attends over the same cached rows.
//
//  * latent_norm        : splits the down projections of a row [query latent | latent | head gates], RMS-norms the two
//                         latents, writes the latent to its cache row, and the sigmoid of the gates.
//  * head_product       : out[t, n, :] = B_n a[t, n, :] (optionally times a gate per (t, n)): the query-side and
//                         output-side products, one small matrix per head, weights streamed once.
//  * latent_attend_tc   : attention of single query rows on tcgen05 (rank a multiple of 128 up to 512), see below.
//  * latent_attend_mma  : the same on mma.sync for the other ranks, 16 or 32 heads per CTA. Latent rows come in tiles
//                         of 32 tokens by cp.async, double or triple buffered; a tile is both K and V. Every warp owns
//                         a slice of the rank columns. The visible range can be cut over CTAs, with
//                         latent_merge joining the parts.
//  * latent_attend_rows : the same for any rank and type on plain FMAs (fp32 models, ranks beyond 512).
// A query row is (sequence slot, position): its keys are the `window` tokens that end with itself (window <= 0: all up to itself), so
// decoding, continued prompts and mixed batches are the same call.
// Cache rows have a pitch of `rp` >= rank elements whose tail is zero; slots are block * block_size + offset.
#include "host_common.h"
#include "ptx.cuh"

namespace icb {

// ------------------------------------------------------------------------------------------------ latent_norm
constexpr int kLatentNormThreads = 128;

template <typename T>
__device__ __forceinline__ void store4(T* p, float a, float b, float c, float d);
template <>
__device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <>
__device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(a, b), pack_bf16x2(c, d));
}

// WPR warps per row: 1 for many rows (no block-wide step), 4 for a few. VEC 4 needs q_rank, rank, ldq and rp to be
// multiples of 4 (ldz always is).
template <typename T, int WPR, int VEC>
__global__ void __launch_bounds__(kLatentNormThreads)
latent_norm_kernel(const float* __restrict__ z, long long ldz, const float* __restrict__ wq,
                   const float* __restrict__ wc, T* __restrict__ cq, int ldq, T* __restrict__ c,
                   T* __restrict__ cache, const long long* __restrict__ slots, float* __restrict__ gate, int rows,
                   int q_rank, int rank, int rp, int heads, float eps) {
  constexpr int kRowsPerBlock = kLatentNormThreads / 32 / WPR;
  constexpr int kStep = WPR * 32 * VEC;
  __shared__ float red[2][kLatentNormThreads / 32];
  const int row = blockIdx.x * kRowsPerBlock + (WPR == 1 ? threadIdx.x >> 5 : 0);
  const int first = (WPR == 1 ? threadIdx.x & 31 : threadIdx.x) * VEC;
  if (row >= rows) return;                               // whole warps (WPR 1) or whole blocks
  const float* zq = z + (size_t)row * ldz;
  const float* zc = zq + q_rank;
  const float* zg = zc + rank;
  auto square_sum = [&](const float* p, int n) {
    float s = 0.f;
#pragma unroll 4
    for (int i = first; i < n; i += kStep) {
      if constexpr (VEC == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p + i);
        s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      } else {
        s += p[i] * p[i];
      }
    }
    return warp_sum(s);
  };
  float sq = square_sum(zq, q_rank), sc = square_sum(zc, rank);
  if constexpr (WPR > 1) {
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sc; }
    __syncthreads();
    sq = sc = 0.f;
#pragma unroll
    for (int w = 0; w < WPR; ++w) { sq += red[0][w]; sc += red[1][w]; }
  }
  const float iq = 1.f / sqrtf(sq / (float)q_rank + eps);
  const float ic = 1.f / sqrtf(sc / (float)rank + eps);
  // scaled row with a zero tail up to `width`, to one or two destinations
  auto emit = [&](const float* p, const float* w, float inv, int n, int width, T* d0, T* d1) {
#pragma unroll 4
    for (int i = first; i < width; i += kStep) {
      if constexpr (VEC == 4) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < n) {
          const float4 x = *reinterpret_cast<const float4*>(p + i);
          const float4 g = *reinterpret_cast<const float4*>(w + i);
          v = make_float4(x.x * inv * g.x, x.y * inv * g.y, x.z * inv * g.z, x.w * inv * g.w);
        }
        if (d0 != nullptr) store4<T>(d0 + i, v.x, v.y, v.z, v.w);
        if (d1 != nullptr) store4<T>(d1 + i, v.x, v.y, v.z, v.w);
      } else {
        const T v = static_cast<T>(i < n ? p[i] * inv * w[i] : 0.f);
        if (d0 != nullptr) d0[i] = v;
        if (d1 != nullptr) d1[i] = v;
      }
    }
  };
  emit(zq, wq, iq, q_rank, ldq, cq + (size_t)row * ldq, nullptr);
  const long long slot = cache != nullptr ? slots[row] : -1;
  emit(zc, wc, ic, rank, rp, slot >= 0 ? cache + (size_t)slot * rp : nullptr,
       c != nullptr ? c + (size_t)row * rp : nullptr);
  for (int i = first / VEC; i < heads; i += WPR * 32)
    gate[(size_t)row * heads + i] = 1.f / (1.f + expf(-zg[i]));
}

template <typename T>
static int launch_latent_norm(const float* z, long long ldz, const float* wq, const float* wc, void* cq, int ldq,
                              void* c, void* cache, const long long* slots, float* gate, int rows, int q_rank, int rank,
                              int rp, int heads, float eps, cudaStream_t st) {
  const bool wide = q_rank % 4 == 0 && rank % 4 == 0 && ldq % 4 == 0 && rp % 4 == 0 && ldz % 4 == 0;
#define ICB_LN(WPR, VEC)                                                                                              \
  latent_norm_kernel<T, WPR, VEC><<<WPR == 1 ? (rows + 3) / 4 : rows, kLatentNormThreads, 0, st>>>(                   \
      z, ldz, wq, wc, reinterpret_cast<T*>(cq), ldq, reinterpret_cast<T*>(c), reinterpret_cast<T*>(cache), slots, gate, \
      rows, q_rank, rank, rp, heads, eps)
  if (rows >= 8 * num_sms()) {
    if (wide) ICB_LN(1, 4);
    else ICB_LN(1, 1);
  } else {
    if (wide) ICB_LN(4, 4);
    else ICB_LN(4, 1);
  }
#undef ICB_LN
  return check_launch("latent_norm_kernel");
}

// ----------------------------------------------------------------------------------------------- head_product
__device__ __forceinline__ void mma_bf16_16816(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3,
                                               uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// a: [rows, heads * K], b: [heads, N, K], out: [rows, heads * N]; K a multiple of 32, N of 16. A CTA makes 32 output
// columns of MT * 16 rows, its W warps taking turns along K and meeting in shared memory: a few rows against many small
// matrices is bound by latency, so the K loop of a warp is kept short and the grid large. The order of the contraction
// index inside a group of 32 is free as long as both operands use the same one, so lane (r, c) takes elements
// [8 c, 8 c + 8) of its rows with one 16-byte load each, which fill the fragments of two consecutive k-steps.
template <int MT, int W>
__global__ void __launch_bounds__(W * 32)
head_product_mma_kernel(const uint16_t* __restrict__ a, const uint16_t* __restrict__ b, uint16_t* __restrict__ out,
                        const float* __restrict__ gate, int rows, int heads, int K, int N) {
  constexpr int kVals = MT * 16;                             // accumulators of a lane: MT x 4 column tiles x 4
  __shared__ float red[4][kVals][32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = lane >> 2, c = lane & 3;
  const int head = blockIdx.y;
  const int n0 = blockIdx.x * 32;
  const int m0 = blockIdx.z * MT * 16;
  const bool wide = n0 + 16 < N;                             // (N is a multiple of 16: the last CTA may have half)
  const long long lda = (long long)heads * K;
  const uint16_t* bp = b + ((size_t)head * N + n0 + r) * K + c * 8;
  const uint16_t* ap = a + (size_t)head * K + c * 8;
  float acc[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int k = warp * 32; k < K; k += W * 32) {
    uint4 u[4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
      u[j] = (j < 2 || wide) ? *reinterpret_cast<const uint4*>(bp + (size_t)j * 8 * K + k) : zero;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int ra = m0 + m * 16 + r;
      const uint4 v0 = ra < rows ? *reinterpret_cast<const uint4*>(ap + (size_t)ra * lda + k) : zero;
      const uint4 v1 = ra + 8 < rows ? *reinterpret_cast<const uint4*>(ap + (size_t)(ra + 8) * lda + k) : zero;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        mma_bf16_16816(acc[m][j], v0.x, v1.x, v0.y, v1.y, u[j].x, u[j].y);
        mma_bf16_16816(acc[m][j], v0.z, v1.z, v0.w, v1.w, u[j].z, u[j].w);
      }
    }
  }
  auto put = [&](int w) {
#pragma unroll
    for (int i = 0; i < kVals; ++i) red[w][i][lane] = acc[i >> 4][(i >> 2) & 3][i & 3];
  };
  if constexpr (W == 8) {
    if (warp >= 4) put(warp - 4);
    __syncthreads();
    if (warp < 4) {
#pragma unroll
      for (int i = 0; i < kVals; ++i) acc[i >> 4][(i >> 2) & 3][i & 3] += red[warp][i][lane];
    }
    __syncthreads();
  }
  if (warp < 4) put(warp);
  __syncthreads();
#pragma unroll
  for (int p = warp; p < MT * 8; p += W) {                   // p = (m, j, half): a pair of neighbouring columns per lane
    const int m = p >> 3, j = (p >> 1) & 3, half = p & 1;
    const int row = m0 + m * 16 + half * 8 + r;
    if (row < rows && (j < 2 || wide)) {
      float lo = 0.f, hi = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        lo += red[w][m * 16 + j * 4 + half * 2][lane];
        hi += red[w][m * 16 + j * 4 + half * 2 + 1][lane];
      }
      const float gt = gate != nullptr ? gate[(size_t)row * heads + head] : 1.f;
      *reinterpret_cast<uint32_t*>(out + ((size_t)row * heads + head) * N + n0 + 8 * j + 2 * c) =
          pack_bf16x2(lo * gt, hi * gt);
    }
  }
}

template <int MT>
static void launch_head_product(const uint16_t* a, const uint16_t* b, uint16_t* out, const float* gate, int rows,
                                int heads, int K, int N, cudaStream_t st) {
  const dim3 grid((N + 31) / 32, heads, (rows + MT * 16 - 1) / (MT * 16));
  if (K >= 256) head_product_mma_kernel<MT, 8><<<grid, 256, 0, st>>>(a, b, out, gate, rows, heads, K, N);
  else head_product_mma_kernel<MT, 4><<<grid, 128, 0, st>>>(a, b, out, gate, rows, heads, K, N);
}

// The same product in fp32: one CTA per (row, head), a warp per output value.
__global__ void __launch_bounds__(128)
head_product_f32_kernel(const float* __restrict__ a, const float* __restrict__ b, float* __restrict__ out,
                        const float* __restrict__ gate, int rows, int heads, int K, int N) {
  const int row = blockIdx.x, head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* ar = a + ((size_t)row * heads + head) * K;
  const float gt = gate != nullptr ? gate[(size_t)row * heads + head] : 1.f;
  for (int n = warp; n < N; n += 4) {
    const float* br = b + ((size_t)head * N + n) * K;
    float s = 0.f;
    for (int k = lane; k < K; k += 32) s += ar[k] * br[k];
    s = warp_sum(s);
    if (lane == 0) out[((size_t)row * heads + head) * N + n] = s * gt;
  }
}

// ----------------------------------------------------------------------------------------- latent_attend_rows
struct LatentAttendArgs {
  const void* q;              // [rows, heads, rp]
  const void* cache;          // [slots, rp]
  const int* block_table;     // [sequences, max_blocks]
  const int* row_seq;         // [rows]
  const int* row_pos;         // [rows]
  void* out;                  // [rows, heads, rp]
  float* part;                // [rows, heads, nsplit, rp + 2] when nsplit > 1
  int rows, heads, rp, block_size, max_blocks, window, nsplit;
  float scale;
};

constexpr int kLrChunk = 128;    // keys per pass; one thread per key in the softmax

template <typename T>
__global__ void __launch_bounds__(kLrChunk) latent_attend_rows_kernel(const LatentAttendArgs a) {
  extern __shared__ __align__(16) float lr_smem[];      // q [rp], o [rp]
  __shared__ float s_p[kLrChunk];
  __shared__ float s_red[2][kLrChunk / 32];
  __shared__ const T* s_row[kLrChunk];
  const int row = blockIdx.x, head = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sq = lr_smem;
  float* so = lr_smem + a.rp;
  const T* q = reinterpret_cast<const T*>(a.q) + ((size_t)row * a.heads + head) * a.rp;
  for (int i = threadIdx.x; i < a.rp; i += kLrChunk) {
    sq[i] = static_cast<float>(q[i]) * a.scale;
    so[i] = 0.f;
  }
  const int pos = a.row_pos[row];
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int* bt = a.block_table + (size_t)a.row_seq[row] * a.max_blocks;
  float m = -INFINITY, l = 0.f;
  for (int t0 = lo; t0 <= pos; t0 += kLrChunk) {
    const int n = min(kLrChunk, pos - t0 + 1);
    __syncthreads();
    if ((int)threadIdx.x < n) {
      const int tok = t0 + threadIdx.x;
      s_row[threadIdx.x] = reinterpret_cast<const T*>(a.cache) +
                           ((size_t)bt[tok / a.block_size] * a.block_size + tok % a.block_size) * a.rp;
    }
    __syncthreads();
    for (int k = warp; k < n; k += kLrChunk / 32) {
      const T* cr = s_row[k];
      float s = 0.f;
      for (int i = lane; i < a.rp; i += 32) s += sq[i] * static_cast<float>(cr[i]);
      s = warp_sum(s);
      if (lane == 0) s_p[k] = s;
    }
    __syncthreads();
    const float s = (int)threadIdx.x < n ? s_p[threadIdx.x] : -INFINITY;
    float mx = s;
#pragma unroll
    for (int off = 16; off; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
    if (lane == 0) s_red[0][warp] = mx;
    __syncthreads();
    mx = m;
#pragma unroll
    for (int w = 0; w < kLrChunk / 32; ++w) mx = fmaxf(mx, s_red[0][w]);
    const float corr = m == -INFINITY ? 0.f : expf(m - mx);
    const float p = (int)threadIdx.x < n ? expf(s - mx) : 0.f;
    s_p[threadIdx.x] = p;
    const float ps = warp_sum(p);
    if (lane == 0) s_red[1][warp] = ps;
    __syncthreads();
    l *= corr;
#pragma unroll
    for (int w = 0; w < kLrChunk / 32; ++w) l += s_red[1][w];
    m = mx;
    for (int i = threadIdx.x; i < a.rp; i += kLrChunk) {
      float o = so[i] * corr;
      for (int k = 0; k < n; ++k) o += s_p[k] * static_cast<float>(s_row[k][i]);
      so[i] = o;
    }
  }
  T* out = reinterpret_cast<T*>(a.out) + ((size_t)row * a.heads + head) * a.rp;
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int i = threadIdx.x; i < a.rp; i += kLrChunk) out[i] = static_cast<T>(so[i] * inv);
}

// ------------------------------------------------------------------------------------------ latent_attend_mma
constexpr int kLmTok = 32;

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// 16 bytes global -> shared; zeros when `ok` is false (the source is not read then)
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int NT, int MT>   // rp = 64 * NT, MT * 16 heads per CTA
struct LmSmem {
  static constexpr int kRp = 64 * NT;
  static constexpr int kWarps = 4;
  static constexpr int kCols = kRp / kWarps;
  static constexpr int kPitch = kRp + 8;                   // rows 16 bytes apart modulo 128: ldmatrix without conflicts
  static constexpr int kStages = NT <= 4 ? 3 : 2;
  static constexpr int tile_bytes = kLmTok * kPitch * 2;
  static constexpr int s_off = kStages * tile_bytes;
  static constexpr int kSPitch = kLmTok + 8;               // float pairs of a fragment row land in distinct banks
  static constexpr int s_bytes = kWarps * MT * 16 * kSPitch * 4;
  static constexpr int p_off = s_off + s_bytes;
  static constexpr int kPPitch = kLmTok + 8;
  static constexpr int p_bytes = MT * 16 * kPPitch * 2;
  static constexpr int row_off = p_off + p_bytes;          // corr, m, l: MT * 16 floats each
  static constexpr int total = row_off + 3 * MT * 16 * 4;
};

// A warp owns a slice of the rank columns in both products. Its slice of Q stays in registers; S = Q C^T is the sum
// of the slices' parts, which meet in shared memory; O += P C needs nothing from the other warps but P.
template <int NT, int MT>
__global__ void __launch_bounds__(LmSmem<NT, MT>::kWarps * 32, 2) latent_attend_mma_kernel(const LatentAttendArgs a) {
  using L = LmSmem<NT, MT>;
  constexpr int kRows = MT * 16;
  constexpr int kWarps = L::kWarps, kThreads = kWarps * 32;
  constexpr int kSteps = L::kCols / 16, kOutTiles = L::kCols / 8;      // k-steps of S, 8-column tiles of O
  extern __shared__ __align__(128) uint8_t lm_smem[];
  const int row = blockIdx.x, h0 = blockIdx.y * kRows, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int fr = lane >> 2, fc = lane & 3;                   // fragment row / column pair of this lane
  float* sS = reinterpret_cast<float*>(lm_smem + L::s_off);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(lm_smem + L::p_off);
  float* s_corr = reinterpret_cast<float*>(lm_smem + L::row_off);
  float* s_m = s_corr + kRows;
  float* s_l = s_m + kRows;
  const uint32_t c_addr = smem_u32(lm_smem);
  const uint32_t p_addr = c_addr + L::p_off;

  const int pos = a.row_pos[row];
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int tiles = (pos - lo + kLmTok) / kLmTok;            // ceil((pos - lo + 1) / 32)
  const int per = (tiles + a.nsplit - 1) / a.nsplit;
  const int t_begin = split * per, t_end = min(tiles, t_begin + per);
  const int* bt = a.block_table + (size_t)a.row_seq[row] * a.max_blocks;
  const uint16_t* cache = reinterpret_cast<const uint16_t*>(a.cache);

  // Eight threads load a token row; a thread's rows (one per kThreads / 8) move on by 32 tokens per tile. Where the
  // next tile's rows are is looked up one tile ahead, so that the copies never wait for the page table.
  constexpr int kLoadRows = kLmTok / (kThreads / 8);
  int next_tok[kLoadRows], next_off[kLoadRows], next_page[kLoadRows], next_blk[kLoadRows];
#pragma unroll
  for (int i = 0; i < kLoadRows; ++i) {
    next_tok[i] = lo + t_begin * kLmTok + (threadIdx.x >> 3) + i * (kThreads / 8);
    next_page[i] = next_tok[i] / a.block_size;
    next_off[i] = next_tok[i] - next_page[i] * a.block_size;
    next_blk[i] = next_tok[i] <= pos ? bt[next_page[i]] : 0;
  }
  auto load_tile = [&](int t) {
    if (t < t_end) {
      const uint32_t stage = c_addr + ((t - t_begin) % L::kStages) * L::tile_bytes;
#pragma unroll
      for (int i = 0; i < kLoadRows; ++i) {
        const bool ok = next_tok[i] <= pos;
        const uint16_t* src = ok ? cache + ((size_t)next_blk[i] * a.block_size + next_off[i]) * L::kRp : cache;
        const uint32_t dst = stage + ((threadIdx.x >> 3) + i * (kThreads / 8)) * (L::kPitch * 2);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int ch = (threadIdx.x & 7) + j * 8;
          cp_async16(dst + ch * 16, src + ch * 8, ok);
        }
        next_tok[i] += kLmTok;
        next_off[i] += kLmTok;
        while (next_off[i] >= a.block_size) { next_off[i] -= a.block_size; ++next_page[i]; }
        if (next_tok[i] <= pos) next_blk[i] = bt[next_page[i]];
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < L::kStages - 1; ++s) load_tile(t_begin + s);

  const int col0 = warp * L::kCols;                          // this warp's rank columns
  uint32_t qf[MT][kSteps][4];
  {
    const uint16_t* q = reinterpret_cast<const uint16_t*>(a.q) + (size_t)row * a.heads * L::kRp + col0 + 2 * fc;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int k = 0; k < kSteps; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int hr = h0 + mt * 16 + fr + (e & 1) * 8;
          qf[mt][k][e] = hr < a.heads
              ? *reinterpret_cast<const uint32_t*>(q + (size_t)hr * L::kRp + k * 16 + (e >> 1) * 8) : 0u;
        }
  }
  float acc[MT][kOutTiles][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < kOutTiles; ++n) acc[mt][n][0] = acc[mt][n][1] = acc[mt][n][2] = acc[mt][n][3] = 0.f;
  constexpr int kOwn = kRows / kWarps;                       // heads whose softmax this warp does
  float m[kOwn], l[kOwn];                                    // m: the same in every lane; l: this lane's share
#pragma unroll
  for (int e = 0; e < kOwn; ++e) { m[e] = -INFINITY; l[e] = 0.f; }
  const float scale_log2 = a.scale * 1.4426950408889634f;
  const uint32_t s_lane = (((lane >> 4) * 8 + (lane & 7)) * L::kPitch + ((lane >> 3) & 1) * 8 + col0) * 2;
  const uint32_t v_lane = (lane * L::kPitch + col0) * 2;

  for (int t = t_begin; t < t_end; ++t) {
    cp_async_wait<L::kStages - 2>();
    __syncthreads();                                         // tile t is in place, everybody is done with tile t - 1
    load_tile(t + L::kStages - 1);
    const uint32_t tile = c_addr + ((t - t_begin) % L::kStages) * L::tile_bytes;
    // ---- this slice's part of the scores, heads x 16 tokens at a time
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float sc[MT][2][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 2; ++n) sc[mt][n][0] = sc[mt][n][1] = sc[mt][n][2] = sc[mt][n][3] = 0.f;
#pragma unroll
      for (int k = 0; k < kSteps; ++k) {
        uint32_t b[4];
        ldsm_x4(b, tile + s_lane + half * 16 * (L::kPitch * 2) + k * 32);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16_16816(sc[mt][0], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[0], b[1]);
          mma_bf16_16816(sc[mt][1], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[2], b[3]);
        }
      }
      float* dst = sS + (warp * kRows + fr) * L::kSPitch + half * 16 + 2 * fc;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* d = dst + mt * 16 * L::kSPitch + n * 8;
          *reinterpret_cast<float2*>(d) = make_float2(sc[mt][n][0], sc[mt][n][1]);
          *reinterpret_cast<float2*>(d + 8 * L::kSPitch) = make_float2(sc[mt][n][2], sc[mt][n][3]);
        }
    }
    __syncthreads();
    // ---- online softmax of this warp's heads; a lane is a token of the tile (the first one is always visible)
    {
      const bool seen = lo + t * kLmTok + lane <= pos;
      float s[kOwn], mx[kOwn];
#pragma unroll
      for (int e = 0; e < kOwn; ++e) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kWarps; ++w) v += sS[(w * kRows + warp * kOwn + e) * L::kSPitch + lane];
        s[e] = mx[e] = seen ? v * scale_log2 : -INFINITY;
      }
#pragma unroll
      for (int off = 16; off; off >>= 1)
#pragma unroll
        for (int e = 0; e < kOwn; ++e) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], off));
#pragma unroll
      for (int e = 0; e < kOwn; ++e) {
        const float top = fmaxf(mx[e], m[e]);
        const float corr = ex2(m[e] - top);
        const float p = ex2(s[e] - top);
        l[e] = l[e] * corr + p;
        m[e] = top;
        sP[(warp * kOwn + e) * L::kPPitch + lane] = __float2bfloat16(p);
        if (lane == 0) s_corr[warp * kOwn + e] = corr;
      }
    }
    __syncthreads();
    // ---- O = O * corr + P C over this warp's columns
    uint32_t pa[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const uint32_t pl = p_addr + ((mt * 16 + (lane & 15)) * L::kPPitch + (lane >> 4) * 8) * 2;
      ldsm_x4(pa[mt][0], pl);
      ldsm_x4(pa[mt][1], pl + 32);
      const float c0 = s_corr[mt * 16 + fr], c1 = s_corr[mt * 16 + fr + 8];
      if (__any_sync(0xffffffffu, c0 != 1.f || c1 != 1.f)) {
#pragma unroll
        for (int n = 0; n < kOutTiles; ++n) {
          acc[mt][n][0] *= c0; acc[mt][n][1] *= c0; acc[mt][n][2] *= c1; acc[mt][n][3] *= c1;
        }
      }
    }
#pragma unroll
    for (int n = 0; n < kOutTiles; ++n) {
      uint32_t b[4];
      ldsm_x4_t(b, tile + v_lane + n * 16);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        mma_bf16_16816(acc[mt][n], pa[mt][0][0], pa[mt][0][1], pa[mt][0][2], pa[mt][0][3], b[0], b[1]);
        mma_bf16_16816(acc[mt][n], pa[mt][1][0], pa[mt][1][1], pa[mt][1][2], pa[mt][1][3], b[2], b[3]);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int e = 0; e < kOwn; ++e) {
    const float sum = warp_sum(l[e]);
    if (lane == 0) { s_m[warp * kOwn + e] = m[e]; s_l[warp * kOwn + e] = sum; }
  }
  __syncthreads();
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int hr = mt * 16 + fr + half * 8;
      if (h0 + hr < a.heads) {
        const int col = col0 + 2 * fc;
        const size_t head_row = (size_t)row * a.heads + h0 + hr;
        if (a.nsplit == 1) {
          const float inv = s_l[hr] > 0.f ? 1.f / s_l[hr] : 0.f;
          uint16_t* o = reinterpret_cast<uint16_t*>(a.out) + head_row * L::kRp + col;
#pragma unroll
          for (int n = 0; n < kOutTiles; ++n)
            *reinterpret_cast<uint32_t*>(o + n * 8) =
                pack_bf16x2(acc[mt][n][half * 2] * inv, acc[mt][n][half * 2 + 1] * inv);
        } else {
          float* rec = a.part + (head_row * a.nsplit + split) * (L::kRp + 2);
#pragma unroll
          for (int n = 0; n < kOutTiles; ++n)
            *reinterpret_cast<float2*>(rec + col + n * 8) = make_float2(acc[mt][n][half * 2], acc[mt][n][half * 2 + 1]);
          if (warp == 0 && fc == 0) *reinterpret_cast<float2*>(rec + L::kRp) = make_float2(s_m[hr], s_l[hr]);
        }
      }
    }
}

// ------------------------------------------------------------------------------------------- latent_attend_tc
// tcgen05 form, 16 or 32 heads (HN) of one query row per CTA, one CTA per SM. Heads are far fewer than the 128 rows of
// an MMA, so both products run transposed, with the cached rows as the M side and the heads as the N side:
//   S^T [128 tokens, HN]   = C [128 tokens, rank] Q^T              A = C K-major,  B = Q [HN, rank] K-major
//   O^T [rank, HN]        += C^T [rank, 128 tokens] P^T            A = C MN-major, B = P [HN, tokens] K-major
// and one copy of a tile of C in shared memory serves both. It arrives through TMA in pairs of 64-column chunks
// ([128 tokens][64], 128-byte swizzle; a box has 16 to 128 rows, the most that page borders allow, and pages of 64 and
// more tokens keep the number of copies small); a
// ring of five pairs holds one tile of rank 512 plus the next tile's first pair, and a block of O^T gives its pair back
// as soon as its MMAs are done. Warp 0 loads, warp 1 issues MMAs, warps 2-5 do the softmax: S^T comes out of TMEM one
// token per lane, is transposed inside the warp through shared memory to one head per lane, and the four warps exchange
// only their maxima. The accumulator is rescaled when a head's maximum grows by more than 2^8 (exact: the
// normalisation uses the same reference), so TMEM is rarely read back. Every wait is bounded.
constexpr int kLtThreads = 192;
constexpr int kLtPairs = 5;
constexpr int kLtTok = 128;

template <int NP, int HN>   // rank = 128 * NP
struct LtSmem {
  static constexpr int kRank = 128 * NP;
  static constexpr int pair_bytes = 2 * kLtTok * 128;
  static constexpr int q_off = kLtPairs * pair_bytes;
  static constexpr int q_chunk = HN * 128;
  static constexpr int p_off = q_off + 2 * NP * q_chunk;
  static constexpr int t_off = p_off + 2 * q_chunk;
  static constexpr int kTPitch = 33;
  static constexpr int x_off = t_off + kLtTok * kTPitch * 4;      // maxima [2][4][32], sums [4][32]
  static constexpr int bar_off = x_off + 3 * 4 * 32 * 4;
  static constexpr int total = bar_off + 128 + 1024;              // manual 1 KiB alignment
  static constexpr int tmem_s = 128;                              // O^T in columns [0, NP * HN), S^T behind
};

template <int NP, int HN>
__global__ void __launch_bounds__(kLtThreads, 1)
latent_attend_tc_kernel(const __grid_constant__ CUtensorMap tmC, const LatentAttendArgs a, int box_log2, int* status) {
  using L = LtSmem<NP, HN>;
  extern __shared__ __align__(1024) uint8_t lt_smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem + L::q_off;
  uint8_t* sP = smem + L::p_off;
  float* sT = reinterpret_cast<float*>(smem + L::t_off);
  float* sX = reinterpret_cast<float*>(smem + L::x_off);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::bar_off);
  uint64_t* full = bars;                 // kLtPairs
  uint64_t* empty = bars + kLtPairs;     // kLtPairs
  uint64_t* s_full = bars + 2 * kLtPairs;
  uint64_t* p_full = s_full + 1;
  uint64_t* o_full = s_full + 2;
  uint64_t* q_full = s_full + 3;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(s_full + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int row = blockIdx.x, h0 = blockIdx.y * HN, split = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pos = a.row_pos[row];
  const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  const int box_rows = 1 << box_log2;
  const int base = lo & ~(box_rows - 1);                      // tiles start on a box
  const int tiles = (pos - base) / kLtTok + 1;
  const int per = (tiles + a.nsplit - 1) / a.nsplit;
  const int t_begin = split * per, t_end = min(tiles, t_begin + per);
  const size_t head_row0 = (size_t)row * a.heads + h0;
  const int heads = min(HN, a.heads - h0);

  if (t_begin >= t_end) {                                     // an empty range (only with several)
    for (int h = 0; h < heads; ++h) {
      float* rec = a.part + ((head_row0 + h) * a.nsplit + split) * (L::kRank + 2);
      for (int i = threadIdx.x; i < L::kRank + 2; i += kLtThreads) rec[i] = i == L::kRank ? -INFINITY : 0.f;
    }
    return;
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < kLtPairs; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 1);
    }
    mbar_init(s_full, 1);
    mbar_init(p_full, 128);
    mbar_init(o_full, 1);
    mbar_init(q_full, 128);
    *abort_flag = 0;
    fence_mbar_init();
    tma_prefetch_desc(&tmC);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_o = *tmem_slot;
  const uint32_t tmem_s = tmem_o + L::tmem_s;
  const int n_tiles = t_end - t_begin;

  if (warp == 0) {
    // ----------------------------- loads: lane = (chunk of the pair, box of the tile) -----------------------------
    const int* bt = a.block_table + (size_t)a.row_seq[row] * a.max_blocks;
    const int nb_log2 = 7 - box_log2, nb = 1 << nb_log2;      // boxes per chunk
    const int box = lane & (nb - 1), chunk = (lane >> nb_log2) & 1;
    // The ring asks for a tile 256 bytes of a row at a time, which DRAM serves poorly; whole boxes (contiguous rows) are
    // brought into L2 ahead of it.
    auto prefetch = [&](int t) {
      const int tok = base + (t_begin + t) * kLtTok + box * box_rows;
      if (t < n_tiles && lane < nb && tok <= pos) {
        const int page = tok / a.block_size;
        const uint16_t* src = reinterpret_cast<const uint16_t*>(a.cache) +
                              ((size_t)bt[page] * a.block_size + (tok - page * a.block_size)) * L::kRank;
        asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(src), "r"(box_rows * L::kRank * 2) : "memory");
      }
    };
    int idx = 0;
    for (int t = 0; t < n_tiles; ++t) {
      // boxes past the position repeat its own one: finite values for keys whose weight is zero
      const int tok = min(base + (t_begin + t) * kLtTok + box * box_rows, pos & ~(box_rows - 1));
      const int page = tok / a.block_size;
      const int y = bt[page] * a.block_size + (tok - page * a.block_size);
      for (int j = 0; j < NP; ++j, ++idx) {
        const int s = idx % kLtPairs;
        mbar_wait(&empty[s], ((idx / kLtPairs) & 1) ^ 1, abort_flag, status, kTimeoutSmemEmpty);
        if (lane == 0) mbar_expect_tx(&full[s], L::pair_bytes);
        __syncwarp();
        if (lane < 2 * nb)
          tma_load_2d(smem + s * L::pair_bytes + chunk * (kLtTok * 128) + box * (box_rows * 128), &tmC, &full[s],
                      (2 * j + chunk) * 64, y);
        if (j == (NP - 1) / 2) prefetch(t + 2);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    // The whole warp walks the loops, so that descriptors stay in uniform registers; one lane issues. Descriptors hold
    // addresses in units of sixteen bytes and shared memory ends below their field, so a step is an addition.
    const bool leader = elect_one() != 0;
    const uint32_t idesc_s = umma_idesc(128, HN, 1, 0, 0);
    const uint32_t idesc_o = umma_idesc(128, HN, 1, 1, 0);
    const uint64_t c_k = umma_desc_sw128(smem_u32(smem), 16, 1024);                  // C as the K-major operand
    const uint64_t c_mn = umma_desc_sw128(smem_u32(smem), kLtTok * 128, 1024);       // C as the MN-major operand
    const uint64_t q_desc = umma_desc_sw128(smem_u32(sQ), 16, 1024);
    const uint64_t p_desc = umma_desc_sw128(smem_u32(sP), 16, 1024);
    mbar_wait(q_full, 0, abort_flag, status, kTimeoutLocalFlag);
    int idx = 0;
    for (int t = 0; t < n_tiles; ++t) {
      for (int j = 0; j < NP; ++j) {
        const int s = (idx + j) % kLtPairs;
        mbar_wait(&full[s], ((idx + j) / kLtPairs) & 1, abort_flag, status, kTimeoutSmemFull);
        tc_fence_after();
        const uint64_t ad = c_k + (uint64_t)(s * (L::pair_bytes >> 4));
        const uint64_t bd = q_desc + (uint64_t)(j * (2 * L::q_chunk >> 4));
        if (leader) {
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_ss(tmem_s, ad + (((k >> 2) * (kLtTok * 128) + (k & 3) * 32) >> 4),
                    bd + (((k >> 2) * L::q_chunk + (k & 3) * 32) >> 4), idesc_s, (j > 0 || k > 0) ? 1u : 0u);
        }
        __syncwarp();
      }
      if (leader) umma_commit(s_full);
      __syncwarp();
      mbar_wait(p_full, t & 1, abort_flag, status, kTimeoutLocalFlag);
      tc_fence_after();
      for (int j = 0; j < NP; ++j, ++idx) {
        const int s = idx % kLtPairs;
        const uint64_t ad = c_mn + (uint64_t)(s * (L::pair_bytes >> 4));
        if (leader) {
#pragma unroll
          for (int k = 0; k < kLtTok / 16; ++k)
            umma_ss(tmem_o + j * HN, ad + (k * 2048 >> 4), p_desc + (((k >> 2) * L::q_chunk + (k & 3) * 32) >> 4), idesc_o,
                    (t > 0 || k > 0) ? 1u : 0u);
          umma_commit(&empty[s]);
        }
        __syncwarp();
      }
    }
    if (leader) umma_commit(o_full);
    __syncwarp();
  } else {
    // ----------------------------------------- softmax and epilogue -----------------------------------------
    const int q = warp & 3;                                   // TMEM lanes 32 q .. 32 q + 31
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    const int head = lane % HN;                               // of this lane after the transposition
    const int sub = HN == 32 ? 0 : (lane >> 4) * 16;          // its HN tokens of the warp's 32 start here
    float* my = sT + q * 32 * L::kTPitch;
    const float scale_log2 = a.scale * 1.4426950408889634f;
    constexpr int kGroups = (NP * HN + 31) / 32;              // O^T in groups of 32 columns
    {
      // Q in the K-major swizzled layout: 64-column chunks of [HN rows][128 bytes]; all loads of a thread in flight
      const uint16_t* qg = reinterpret_cast<const uint16_t*>(a.q) + head_row0 * L::kRank;
      constexpr int kPieces = L::kRank / 8, kEach = HN * kPieces / 128;
      uint4 u[kEach];
#pragma unroll
      for (int i = 0; i < kEach; ++i) {
        const int hr = (i * 128 + (int)threadIdx.x - 64) / kPieces, piece = (i * 128 + (int)threadIdx.x - 64) % kPieces;
        u[i] = hr < heads ? *reinterpret_cast<const uint4*>(qg + (size_t)hr * L::kRank + piece * 8)
                          : make_uint4(0u, 0u, 0u, 0u);
      }
#pragma unroll
      for (int i = 0; i < kEach; ++i) {
        const int hr = (i * 128 + (int)threadIdx.x - 64) / kPieces, piece = (i * 128 + (int)threadIdx.x - 64) % kPieces;
        *reinterpret_cast<uint4*>(sQ + (piece >> 3) * L::q_chunk + hr * 128 + (((piece & 7) ^ (hr & 7)) << 4)) = u[i];
      }
      fence_proxy_async_smem();
      mbar_arrive(q_full);
    }
    float m_ref = -INFINITY, l = 0.f;
    for (int t = 0; t < n_tiles; ++t) {
      mbar_wait(s_full, t & 1, abort_flag, status, kTimeoutTmemFull);
      tc_fence_after();
      {
        uint32_t r[HN];
        if constexpr (HN == 32) tmem_ld_32x32(tmem_s + lane_off, r);
        else tmem_ld_32x16(tmem_s + lane_off, r);
        tmem_ld_wait();
#pragma unroll
        for (int h = 0; h < HN; ++h) my[lane * L::kTPitch + h] = __uint_as_float(r[h]);
      }
      __syncwarp();
      const int tok0 = base + (t_begin + t) * kLtTok + q * 32 + sub;
      float v[HN], mx;
#pragma unroll
      for (int i = 0; i < HN; ++i) v[i] = my[(sub + i) * L::kTPitch + head] * scale_log2;
      if (base + (t_begin + t) * kLtTok < lo || base + (t_begin + t + 1) * kLtTok > pos + 1) {   // a border tile
#pragma unroll
        for (int i = 0; i < HN; ++i)
          if (tok0 + i < lo || tok0 + i > pos) v[i] = -INFINITY;
      }
      {
        float m4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
        for (int i = 4; i < HN; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
        mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3]));
      }
      if constexpr (HN == 16) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 16));
      float* x = sX + (t & 1) * 128;
      if (sub == 0) x[q * 32 + head] = mx;
      named_barrier(1, 128);
      mx = fmaxf(fmaxf(x[head], x[32 + head]), fmaxf(x[64 + head], x[96 + head]));   // the same in all four warps
      const bool grow = mx > m_ref + 8.f;                     // always in the first tile
      float factor = 1.f;
      if (grow) {
        factor = ex2(m_ref - mx);
        m_ref = mx;
        l *= factor;
      }
      if (t > 0 && __any_sync(0xffffffffu, grow)) {           // (S^T of this tile is behind O^T of the last: complete)
#pragma unroll
        for (int g = 0; g < kGroups; ++g) {
          uint32_t o[32];
          tmem_ld_32x32(tmem_o + lane_off + g * 32, o);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i)
            o[i] = __float_as_uint(__uint_as_float(o[i]) * __shfl_sync(0xffffffffu, factor, i % HN));
          tmem_st_32x32(tmem_o + lane_off + g * 32, o);
        }
        tmem_st_wait();
      }
      const int tile_tok = q * 32 + sub;
      uint8_t* prow = sP + (tile_tok >> 6) * L::q_chunk + head * 128;
      float l4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < HN; i += 8) {
        float p[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          p[e] = ex2(v[i + e] - m_ref);
          l4[e & 3] += p[e];
        }
        uint4 u;
        u.x = pack_bf16x2(p[0], p[1]); u.y = pack_bf16x2(p[2], p[3]);
        u.z = pack_bf16x2(p[4], p[5]); u.w = pack_bf16x2(p[6], p[7]);
        const int piece = ((tile_tok + i) & 63) >> 3;
        *reinterpret_cast<uint4*>(prow + ((piece ^ (head & 7)) << 4)) = u;
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(p_full);
      l += (l4[0] + l4[1]) + (l4[2] + l4[3]);
    }
    mbar_wait(o_full, 0, abort_flag, status, kTimeoutTmemFull);
    tc_fence_after();
    if constexpr (HN == 16) l += __shfl_xor_sync(0xffffffffu, l, 16);
    float* sl = sX + 256;
    if (sub == 0) sl[q * 32 + head] = l;
    named_barrier(1, 128);
    l = sl[head] + sl[32 + head] + sl[64 + head] + sl[96 + head];
    const float inv = l > 0.f ? 1.f / l : 0.f;
#pragma unroll
    for (int g = 0; g < kGroups; ++g) {
      uint32_t o[32];
      tmem_ld_32x32(tmem_o + lane_off + g * 32, o);
      tmem_ld_wait();
#pragma unroll
      for (int i = 0; i < 32; ++i) {
        const int col = g * 32 + i;
        const int h = i % HN, rank = (col / HN) * 128 + q * 32 + lane;
        if (a.nsplit == 1) {
          const float w = __shfl_sync(0xffffffffu, inv, h);
          if (col < NP * HN && h < heads)
            reinterpret_cast<__nv_bfloat16*>(a.out)[(head_row0 + h) * L::kRank + rank] =
                __float2bfloat16(__uint_as_float(o[i]) * w);
        } else {
          if (col < NP * HN && h < heads)
            a.part[((head_row0 + h) * a.nsplit + split) * (L::kRank + 2) + rank] = __uint_as_float(o[i]);
        }
      }
    }
    if (a.nsplit > 1 && q == 0 && sub == 0 && head < heads) {
      float* rec = a.part + ((head_row0 + head) * a.nsplit + split) * (L::kRank + 2) + L::kRank;
      rec[0] = m_ref;
      rec[1] = l;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {                                          // let copies in flight land before the memory is given back
    const long long t0 = clock64();
    while (clock64() - t0 < 2000000) { __nanosleep(1000); }
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_o, 256);
  }
}

template <int NP, int HN>
static int launch_latent_tc_h(const CUtensorMap& tm, const LatentAttendArgs& a, int box_log2, int* status,
                              cudaStream_t st) {
  auto kern = latent_attend_tc_kernel<NP, HN>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LtSmem<NP, HN>::total);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  dim3 grid(a.rows, (a.heads + HN - 1) / HN, a.nsplit);
  kern<<<grid, kLtThreads, LtSmem<NP, HN>::total, st>>>(tm, a, box_log2, status);
  return check_launch("latent_attend_tc_kernel");
}
template <int NP>
static int launch_latent_tc(const LatentAttendArgs& a, long long cache_rows, int* status, cudaStream_t st) {
  CUtensorMap tm;
  const uint64_t dims[2] = {(uint64_t)a.rp, (uint64_t)cache_rows};
  const uint64_t strides[1] = {(uint64_t)a.rp * 2};
  int box_log2 = 4;
  while (box_log2 < 7 && a.block_size % (2 << box_log2) == 0) ++box_log2;
  const uint32_t box[2] = {64, 1u << box_log2};
  const int rc = make_tmap(&tm, kBF16, 2, a.cache, dims, strides, box, true);
  if (rc) return rc;
  return a.heads > 16 ? launch_latent_tc_h<NP, 32>(tm, a, box_log2, status, st)
                      : launch_latent_tc_h<NP, 16>(tm, a, box_log2, status, st);
}

// Joins the parts of one (row, head): running maxima are in the log2 domain; an empty part has max -inf and sum 0. A
// thread makes four output values; four parts at a time have all their loads in flight together.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part, uint16_t* __restrict__ out, int rp, int nsplit) {
  const size_t head_row = blockIdx.x;
  const float* rec = part + head_row * nsplit * (rp + 2);
  for (int i = threadIdx.x * 4; i < rp; i += 512) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f}, mx = -INFINITY, l = 0.f;
    for (int s0 = 0; s0 < nsplit; s0 += 4) {
      float2 ml[4], v0[4], v1[4];
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const float* r = rec + (size_t)min(s0 + s, nsplit - 1) * (rp + 2);
        ml[s] = *reinterpret_cast<const float2*>(r + rp);
        v0[s] = *reinterpret_cast<const float2*>(r + i);
        v1[s] = *reinterpret_cast<const float2*>(r + i + 2);
        if (s0 + s >= nsplit) ml[s] = make_float2(-INFINITY, 0.f);
      }
      const float top = fmaxf(fmaxf(fmaxf(ml[0].x, ml[1].x), fmaxf(ml[2].x, ml[3].x)), mx);
      if (top == -INFINITY) continue;
      const float keep = exp2f(mx - top);
      mx = top;
      l *= keep;
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[e] *= keep;
#pragma unroll
      for (int s = 0; s < 4; ++s) {
        const float f = exp2f(ml[s].x - top);
        l += f * ml[s].y;
        acc[0] += f * v0[s].x; acc[1] += f * v0[s].y; acc[2] += f * v1[s].x; acc[3] += f * v1[s].y;
      }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    *reinterpret_cast<uint2*>(out + head_row * rp + i) =
        make_uint2(pack_bf16x2(acc[0] * inv, acc[1] * inv), pack_bf16x2(acc[2] * inv, acc[3] * inv));
  }
}

template <int NT, int MT>
static int launch_latent_mma_m(const LatentAttendArgs& a, cudaStream_t st) {
  auto kern = latent_attend_mma_kernel<NT, MT>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LmSmem<NT, MT>::total);
    if (e != cudaSuccess) return -(int)e;
    configured = true;
  }
  dim3 grid(a.rows, (a.heads + MT * 16 - 1) / (MT * 16), a.nsplit);
  kern<<<grid, LmSmem<NT, MT>::kWarps * 32, LmSmem<NT, MT>::total, st>>>(a);
  return check_launch("latent_attend_mma_kernel");
}
template <int NT>
static int launch_latent_mma(const LatentAttendArgs& a, cudaStream_t st) {
  return a.heads > 16 ? launch_latent_mma_m<NT, 2>(a, st) : launch_latent_mma_m<NT, 1>(a, st);
}

}  // namespace icb

using namespace icb;

// z: [rows, ldz] fp32, columns [query latent (q_rank) | latent (rank) | head gates (heads)]. cq: [rows, ldq];
// c (optional): [rows, rp]; cache (optional) with slots [rows] (negative: skip); gate: [rows, heads] fp32.
ICB_API int icb_latent_norm(const float* z, long long ldz, const float* wq, const float* wc, void* cq, int ldq, void* c,
                            void* cache, const long long* slots, float* gate, int rows, int q_rank, int rank, int rp,
                            int heads, float eps, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (q_rank < 1 || rank < 1 || ldq < q_rank || rp < rank || ldz < q_rank + rank + heads) return -2;
  if (cache != nullptr && slots == nullptr) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16)
    return launch_latent_norm<__nv_bfloat16>(z, ldz, wq, wc, cq, ldq, c, cache, slots, gate, rows, q_rank, rank, rp,
                                             heads, eps, st);
  if (dtype == kF32)
    return launch_latent_norm<float>(z, ldz, wq, wc, cq, ldq, c, cache, slots, gate, rows, q_rank, rank, rp, heads, eps,
                                     st);
  return -3;
}

// out[rows, heads, N] = per head: a[rows, heads, K] B[heads, N, K]^T (times gate[rows, heads] when given).
// bf16: K a multiple of 32, N of 16, 16-byte aligned operands.
ICB_API int icb_head_product(const void* a, const void* b, void* out, const float* gate, int rows, int heads, int K,
                             int N, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (heads < 1 || K < 1 || N < 1) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16) {
    if (K % 32 || N % 16) return -2;
    auto A = reinterpret_cast<const uint16_t*>(a);
    auto B = reinterpret_cast<const uint16_t*>(b);
    auto O = reinterpret_cast<uint16_t*>(out);
    if (rows > 64 * 65535) return -2;
    if (rows <= 16) launch_head_product<1>(A, B, O, gate, rows, heads, K, N, st);
    else if (rows <= 32) launch_head_product<2>(A, B, O, gate, rows, heads, K, N, st);
    else launch_head_product<4>(A, B, O, gate, rows, heads, K, N, st);
  } else if (dtype == kF32) {
    head_product_f32_kernel<<<dim3(rows, heads), 128, 0, st>>>(reinterpret_cast<const float*>(a),
                                                               reinterpret_cast<const float*>(b),
                                                               reinterpret_cast<float*>(out), gate, rows, heads, K, N);
  } else {
    return -3;
  }
  return check_launch("head_product_kernel");
}

// Attention of query rows q [rows, heads, rp] over the latent cache; see the head of this file. bf16 with rp a multiple
// of 64 up to 512 runs on tensor cores (tcgen05 for multiples of 128, unless `legacy` asks for mma.sync), optionally cut
// into nsplit ranges with scratch [rows * heads * nsplit * (rp + 2)] floats; everything else on the plain kernel
// (nsplit is ignored). cache_rows: rows of the cache; block_size a multiple of 16.
ICB_API int icb_latent_attend(const void* q, const void* cache, const int* block_table, const int* row_seq,
                              const int* row_pos, void* out, float* scratch, int rows, int heads, int rp, int block_size,
                              int max_blocks, int window, float scale, int nsplit, int dtype, void* stream,
                              long long cache_rows, int* status, int legacy) {
  if (rows <= 0) return 0;
  if (heads < 1 || rp < 1 || block_size < 16 || block_size % 16 || max_blocks < 1 || nsplit < 1) return -2;
  if (dtype != kBF16 && dtype != kF32) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  LatentAttendArgs a;
  a.q = q; a.cache = cache; a.block_table = block_table; a.row_seq = row_seq; a.row_pos = row_pos; a.out = out;
  a.part = scratch; a.rows = rows; a.heads = heads; a.rp = rp; a.block_size = block_size; a.max_blocks = max_blocks;
  a.window = window; a.nsplit = nsplit; a.scale = scale;
  if (dtype == kBF16 && rp % 64 == 0 && rp <= 512) {
    if (nsplit > 1 && scratch == nullptr) return -4;
    int rc = -2;
    if (rp % 128 == 0 && !legacy) {
      switch (rp / 128) {
        case 1: rc = launch_latent_tc<1>(a, cache_rows, status, st); break;
        case 2: rc = launch_latent_tc<2>(a, cache_rows, status, st); break;
        case 3: rc = launch_latent_tc<3>(a, cache_rows, status, st); break;
        case 4: rc = launch_latent_tc<4>(a, cache_rows, status, st); break;
      }
    } else switch (rp / 64) {
      case 1: rc = launch_latent_mma<1>(a, st); break;
      case 2: rc = launch_latent_mma<2>(a, st); break;
      case 3: rc = launch_latent_mma<3>(a, st); break;
      case 4: rc = launch_latent_mma<4>(a, st); break;
      case 5: rc = launch_latent_mma<5>(a, st); break;
      case 6: rc = launch_latent_mma<6>(a, st); break;
      case 7: rc = launch_latent_mma<7>(a, st); break;
      case 8: rc = launch_latent_mma<8>(a, st); break;
    }
    if (rc == 0 && nsplit > 1) {
      latent_merge_kernel<<<rows * heads, 128, 0, st>>>(scratch, reinterpret_cast<uint16_t*>(out), rp, nsplit);
      rc = check_launch("latent_merge_kernel");
    }
    return rc;
  }
  const size_t smem = (size_t)rp * 2 * sizeof(float);
  if (smem > 200 * 1024) return -6;
  if (dtype == kBF16) {
    if (smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(latent_attend_rows_kernel<__nv_bfloat16>,
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return -(int)e;
    }
    latent_attend_rows_kernel<__nv_bfloat16><<<dim3(rows, heads), kLrChunk, smem, st>>>(a);
  } else {
    if (smem > 40 * 1024) {
      cudaError_t e = cudaFuncSetAttribute(latent_attend_rows_kernel<float>,
                                           cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return -(int)e;
    }
    latent_attend_rows_kernel<float><<<dim3(rows, heads), kLrChunk, smem, st>>>(a);
  }
  return check_launch("latent_attend_rows_kernel");
}
