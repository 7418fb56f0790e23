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
//  * latent_attend_mma  : tensor-core attention of single query rows, 16 or 32 heads per CTA. Latent rows come in tiles
//                         of 32 tokens by cp.async, double or triple buffered; a tile is both K and V. Four warps own
//                         a quarter of the rank columns each. The visible range can be cut over CTAs, with
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

constexpr int kHpWarps = 4;

// a: [rows, heads * K], b: [heads, N, K], out: [rows, heads * N]; K a multiple of 32, N of 16. A warp owns 16 output
// columns of MT * 16 rows. The order of the contraction index inside a group of 32 is free as long as both operands
// use the same one, so lane (r, c) takes elements [8 c, 8 c + 8) of its rows with one 16-byte load each, which fill
// the fragments of two consecutive k-steps.
template <int MT>
__global__ void __launch_bounds__(kHpWarps * 32)
head_product_mma_kernel(const uint16_t* __restrict__ a, const uint16_t* __restrict__ b, uint16_t* __restrict__ out,
                        const float* __restrict__ gate, int rows, int heads, int K, int N) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int r = lane >> 2, c = lane & 3;
  const int head = blockIdx.y;
  const int n0 = (blockIdx.x * kHpWarps + warp) * 16;
  if (n0 >= N) return;
  const int m0 = blockIdx.z * MT * 16;
  const long long lda = (long long)heads * K;
  const uint16_t* b0p = b + ((size_t)head * N + n0 + r) * K + c * 8;
  const uint16_t* b1p = b0p + (size_t)8 * K;
  const uint16_t* ap = a + (size_t)head * K + c * 8;
  float acc[MT][2][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j) acc[m][j][0] = acc[m][j][1] = acc[m][j][2] = acc[m][j][3] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll 2
  for (int k = 0; k < K; k += 32) {
    const uint4 u0 = *reinterpret_cast<const uint4*>(b0p + k);
    const uint4 u1 = *reinterpret_cast<const uint4*>(b1p + k);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const int ra = m0 + m * 16 + r;
      const uint4 v0 = ra < rows ? *reinterpret_cast<const uint4*>(ap + (size_t)ra * lda + k) : zero;
      const uint4 v1 = ra + 8 < rows ? *reinterpret_cast<const uint4*>(ap + (size_t)(ra + 8) * lda + k) : zero;
      mma_bf16_16816(acc[m][0], v0.x, v1.x, v0.y, v1.y, u0.x, u0.y);
      mma_bf16_16816(acc[m][0], v0.z, v1.z, v0.w, v1.w, u0.z, u0.w);
      mma_bf16_16816(acc[m][1], v0.x, v1.x, v0.y, v1.y, u1.x, u1.y);
      mma_bf16_16816(acc[m][1], v0.z, v1.z, v0.w, v1.w, u1.z, u1.w);
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = m0 + m * 16 + half * 8 + r;
      if (row < rows) {
        const float gt = gate != nullptr ? gate[(size_t)row * heads + head] : 1.f;
        uint16_t* o = out + ((size_t)row * heads + head) * N + n0 + 2 * c;
#pragma unroll
        for (int j = 0; j < 2; ++j)
          *reinterpret_cast<uint32_t*>(o + 8 * j) = pack_bf16x2(acc[m][j][half * 2] * gt, acc[m][j][half * 2 + 1] * gt);
      }
    }
  }
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
constexpr int kLmThreads = 128;
constexpr int kLmWarps = kLmThreads / 32;
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

template <int NT, int MT>   // rp = 64 * NT, MT * 16 heads per CTA
struct LmSmem {
  static constexpr int kRp = 64 * NT;
  static constexpr int kPitch = kRp + 8;                   // rows 16 bytes apart modulo 128: ldmatrix without conflicts
  static constexpr int kStages = NT <= 4 ? 3 : 2;
  static constexpr int tile_bytes = kLmTok * kPitch * 2;
  static constexpr int s_off = kStages * tile_bytes;
  static constexpr int kSPitch = kLmTok + 8;               // float pairs of a fragment row land in distinct banks
  static constexpr int s_bytes = kLmWarps * MT * 16 * kSPitch * 4;
  static constexpr int p_off = s_off + s_bytes;
  static constexpr int kPPitch = kLmTok + 8;
  static constexpr int p_bytes = MT * 16 * kPPitch * 2;
  static constexpr int row_off = p_off + p_bytes;          // corr, m, l: MT * 16 floats each
  static constexpr int total = row_off + 3 * MT * 16 * 4;
};

// A warp owns a quarter of the rank columns in both products. Its slice of Q stays in registers; S = Q C^T is the sum
// of the four slices' parts, which meet in shared memory; O += P C needs nothing from the other warps but P.
template <int NT, int MT>
__global__ void __launch_bounds__(kLmThreads, 2) latent_attend_mma_kernel(const LatentAttendArgs a) {
  using L = LmSmem<NT, MT>;
  constexpr int kRows = MT * 16;
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

  auto load_tile = [&](int t) {                              // eight threads per token row, sixteen rows at a time
    if (t < t_end) {
      const uint32_t stage = c_addr + ((t - t_begin) % L::kStages) * L::tile_bytes;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int tr = (threadIdx.x >> 3) + half * 16;
        const int tok = lo + t * kLmTok + tr;
        const bool ok = tok <= pos;
        const uint16_t* src = cache;
        if (ok) {
          const int page = tok / a.block_size;
          src = cache + ((size_t)bt[page] * a.block_size + (tok - page * a.block_size)) * L::kRp;
        }
        const uint32_t dst = stage + tr * (L::kPitch * 2);
#pragma unroll
        for (int j = 0; j < NT; ++j) {
          const int ch = (threadIdx.x & 7) + j * 8;
          cp_async16(dst + ch * 16, src + ch * 8, ok);
        }
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < L::kStages - 1; ++s) load_tile(t_begin + s);

  const int col0 = warp * (16 * NT);                         // this warp's rank columns
  uint32_t qf[MT][NT][4];
  {
    const uint16_t* q = reinterpret_cast<const uint16_t*>(a.q) + (size_t)row * a.heads * L::kRp + col0 + 2 * fc;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int k = 0; k < NT; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int hr = h0 + mt * 16 + fr + (e & 1) * 8;
          qf[mt][k][e] = hr < a.heads
              ? *reinterpret_cast<const uint32_t*>(q + (size_t)hr * L::kRp + k * 16 + (e >> 1) * 8) : 0u;
        }
  }
  float acc[MT][2 * NT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < 2 * NT; ++n) acc[mt][n][0] = acc[mt][n][1] = acc[mt][n][2] = acc[mt][n][3] = 0.f;
  constexpr int kOwn = kRows / kLmWarps;                     // heads whose softmax this warp does
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
    // ---- this slice's part of the scores, heads x 32 tokens
    {
      float sc[MT][4][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n) sc[mt][n][0] = sc[mt][n][1] = sc[mt][n][2] = sc[mt][n][3] = 0.f;
#pragma unroll
      for (int k = 0; k < NT; ++k) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          uint32_t b[4];
          ldsm_x4(b, tile + s_lane + half * 16 * (L::kPitch * 2) + k * 32);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma_bf16_16816(sc[mt][2 * half], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[0], b[1]);
            mma_bf16_16816(sc[mt][2 * half + 1], qf[mt][k][0], qf[mt][k][1], qf[mt][k][2], qf[mt][k][3], b[2], b[3]);
          }
        }
      }
      float* dst = sS + (warp * kRows + fr) * L::kSPitch + 2 * fc;
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < 4; ++n) {
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
        for (int w = 0; w < kLmWarps; ++w) v += sS[(w * kRows + warp * kOwn + e) * L::kSPitch + lane];
        s[e] = mx[e] = seen ? v * scale_log2 : -INFINITY;
      }
#pragma unroll
      for (int off = 16; off; off >>= 1)
#pragma unroll
        for (int e = 0; e < kOwn; ++e) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], off));
#pragma unroll
      for (int e = 0; e < kOwn; ++e) {
        const float top = fmaxf(mx[e], m[e]);
        const float corr = exp2f(m[e] - top);
        const float p = exp2f(s[e] - top);
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
        for (int n = 0; n < 2 * NT; ++n) {
          acc[mt][n][0] *= c0; acc[mt][n][1] *= c0; acc[mt][n][2] *= c1; acc[mt][n][3] *= c1;
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 2 * NT; ++n) {
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
          for (int n = 0; n < 2 * NT; ++n)
            *reinterpret_cast<uint32_t*>(o + n * 8) =
                pack_bf16x2(acc[mt][n][half * 2] * inv, acc[mt][n][half * 2 + 1] * inv);
        } else {
          float* rec = a.part + (head_row * a.nsplit + split) * (L::kRp + 2);
#pragma unroll
          for (int n = 0; n < 2 * NT; ++n)
            *reinterpret_cast<float2*>(rec + col + n * 8) = make_float2(acc[mt][n][half * 2], acc[mt][n][half * 2 + 1]);
          if (warp == 0 && fc == 0) *reinterpret_cast<float2*>(rec + L::kRp) = make_float2(s_m[hr], s_l[hr]);
        }
      }
    }
}

// Joins the parts of one (row, head): running maxima are in the log2 domain; an empty part has max -inf and sum 0.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ part, uint16_t* __restrict__ out, int rp, int nsplit) {
  const size_t head_row = blockIdx.x;
  const float* rec = part + head_row * nsplit * (rp + 2);
  float mx = -INFINITY;
  for (int s = 0; s < nsplit; ++s) mx = fmaxf(mx, rec[(size_t)s * (rp + 2) + rp]);
  float l = 0.f;
  for (int s = 0; s < nsplit; ++s) l += rec[(size_t)s * (rp + 2) + rp + 1] * exp2f(rec[(size_t)s * (rp + 2) + rp] - mx);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  for (int i = threadIdx.x * 2; i < rp; i += 256) {
    float a0 = 0.f, a1 = 0.f;
    for (int s = 0; s < nsplit; ++s) {
      const float f = exp2f(rec[(size_t)s * (rp + 2) + rp] - mx);
      const float2 v = *reinterpret_cast<const float2*>(rec + (size_t)s * (rp + 2) + i);
      a0 += f * v.x;
      a1 += f * v.y;
    }
    *reinterpret_cast<uint32_t*>(out + head_row * rp + i) = pack_bf16x2(a0 * inv, a1 * inv);
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
  kern<<<grid, kLmThreads, LmSmem<NT, MT>::total, st>>>(a);
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
    const int gx = (N + 16 * kHpWarps - 1) / (16 * kHpWarps);
    if (rows <= 16)
      head_product_mma_kernel<1><<<dim3(gx, heads, 1), kHpWarps * 32, 0, st>>>(A, B, O, gate, rows, heads, K, N);
    else if (rows <= 32)
      head_product_mma_kernel<2><<<dim3(gx, heads, 1), kHpWarps * 32, 0, st>>>(A, B, O, gate, rows, heads, K, N);
    else {
      const int gz = (rows + 63) / 64;
      if (gz > 65535) return -2;
      head_product_mma_kernel<4><<<dim3(gx, heads, gz), kHpWarps * 32, 0, st>>>(A, B, O, gate, rows, heads, K, N);
    }
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
// of 64 up to 512 runs on tensor cores, optionally cut into nsplit ranges with scratch
// [rows * heads * nsplit * (rp + 2)] floats; everything else on the plain kernel (nsplit is ignored).
ICB_API int icb_latent_attend(const void* q, const void* cache, const int* block_table, const int* row_seq,
                              const int* row_pos, void* out, float* scratch, int rows, int heads, int rp, int block_size,
                              int max_blocks, int window, float scale, int nsplit, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (heads < 1 || rp < 1 || block_size < 1 || max_blocks < 1 || nsplit < 1) return -2;
  if (dtype != kBF16 && dtype != kF32) return -3;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  LatentAttendArgs a;
  a.q = q; a.cache = cache; a.block_table = block_table; a.row_seq = row_seq; a.row_pos = row_pos; a.out = out;
  a.part = scratch; a.rows = rows; a.heads = heads; a.rp = rp; a.block_size = block_size; a.max_blocks = max_blocks;
  a.window = window; a.nsplit = nsplit; a.scale = scale;
  if (dtype == kBF16 && rp % 64 == 0 && rp <= 512) {
    if (nsplit > 1 && scratch == nullptr) return -4;
    int rc = -2;
    switch (rp / 64) {
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
