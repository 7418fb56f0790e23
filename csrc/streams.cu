// Residual streams with learned mixing (hyper-connections), fused with what surrounds them at a sublayer boundary.
//
// A token carries S residual streams x_1 .. x_S (fp32, [T, S, D]). Between two sublayers a row goes through
//   y'   = y * sigmoid(r + rb)                      gate of the finished sublayer's result (optional)
//   x_t <- sum_s mix[s][t] x_s + out[t] y'          write it into the streams, all from the old values
//   u    = sum_s in[s] x_s                          read the next sublayer's input
//   h    = u / sqrt(mean over its group (u^2) + eps) * w      RMS norm in `groups` equal parts
//   hs   = h + (h_prev - h) * shift                 blend with the previous token's h (optional)
// which is one pass here: the streams are read once and written once per sublayer, everything in fp32.
// The first boundary takes x_s = table[token] * scale instead of the write step; the last one has in = 1 and no
// streams to write, and visits only the rows somebody asked for (row_map). Where a pass of a looped block starts, every
// stream also gets a vector of that pass (add) and, if asked for, the embedding row once more.
//
// The previous token's h of a row is, in this order: the carried value of the row handled just before by the same
// CTA; recomputed from the old streams when that row belongs to another CTA (this is why the streams are written to
// a second buffer); or, for the first row a sequence has in this batch, the sequence's state (zeros at position 0).
//
// Warps are assigned to norm groups, a whole number of warps per group (or a loop over groups per warp), so a row
// needs at most one block-wide barrier.
#include "host_common.h"
#include "ptx.cuh"

namespace icb {

constexpr int kMaxStreams = 16;
constexpr int kStreamMaxWarps = 16;

struct StreamArgs {
  const long long* tokens;      // token ids [T] for the embedding rows
  const void* table;            // embedding rows (pitch ld_table) or null; with x_in they are added to the streams
  long long ld_table, table_rows;   // ids outside the table give zeros
  float table_scale;
  const float* add;             // [D], added to every stream, or null
  const float* x_in;            // [rows, S, D] old streams (null at the first boundary)
  float* x_out;                 // [T, S, D] new streams or null
  const void* y;                // finished sublayer's result, pitch ldy
  long long ldy;
  const void* r;                // its gate logits, pitch ldr, or null
  long long ldr;
  const float* rb;              // [D] bias of the gate logits or null
  const float* mix;             // [S, S], [from][to]
  const float* out;             // [S]
  const int* row_map;           // row of x_in / y / r / tokens for output row i, or null
  const float* in;              // [S]
  const float* norm_w;          // [D]
  int groups;
  float eps;
  void* h;                      // [T, ldh]
  void* hs;                     // [T, ldh] or null (no shift)
  long long ldh;
  const float* shift;           // [D]
  const float* prev;            // [slots, D] previous h by sequence slot, read
  float* state;                 // [slots, D] written with the last h of every sequence of the batch
  const int* row_seq;           // [T] sequence slot of a row; rows of a sequence are adjacent and in order
  const int* row_pos;           // [T] position in the sequence
  int T, S, D, rows_per_block;
};

template <typename T, int V>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[V]) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    const float4 u = *reinterpret_cast<const float4*>(p);
    f[0] = u.x; f[1] = u.y; f[2] = u.z; f[3] = u.w;
  } else if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = static_cast<float>(p[i]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&f)[V]) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = static_cast<T>(f[i]);
  }
}

// S_ > 0 fixes the number of streams at compile time; 0 reads it from the arguments. EXTRA: embedding rows or a vector come
// in (always so at the first boundary).
template <typename T, int S_, int V, bool EXTRA>
__global__ void __launch_bounds__(kStreamMaxWarps * 32) stream_boundary_kernel(const StreamArgs a) {
  extern __shared__ __align__(16) float row_smem[];     // u [D], then (with a shift) the previous row's h [D]
  __shared__ float s_mix[kMaxStreams * kMaxStreams], s_out[kMaxStreams], s_in[kMaxStreams];
  __shared__ float s_red[2][kStreamMaxWarps];
  const int S = S_ > 0 ? S_ : a.S;
  constexpr int SMAX = S_ > 0 ? S_ : kMaxStreams;
  const int D = a.D, G = a.groups, gs = D / G;
  float* su = row_smem;
  float* sprev = row_smem + D;
  const bool write_step = !EXTRA || a.x_in != nullptr;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = write_step ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    s_out[i] = write_step ? a.out[i] : 0.f;
    s_in[i] = a.in[i];
  }
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int warps = blockDim.x >> 5;
  const int wpg = warps >= G ? warps / G : 1;           // the launcher makes `warps` a multiple of G when >= G
  const int g_first = warp / wpg, g_step = warps / wpg, sub = warp % wpg;
  const bool shifted = a.hs != nullptr;
  const int r0 = blockIdx.x * a.rows_per_block;
  const int r1 = min(a.T, r0 + a.rows_per_block);
  int r = r0;
  if (shifted && r0 > 0 && r0 < a.T && a.row_seq[r0 - 1] == a.row_seq[r0]) r = r0 - 1;   // for its h only
  int buf = 0;
  for (; r < r1; ++r) {
    const bool emit = r >= r0;
    const long long src = a.row_map != nullptr ? a.row_map[r] : r;
    int seq = 0;
    bool first = false, last = false;
    const float* before = nullptr;
    if (shifted && emit) {
      seq = a.row_seq[r];
      first = r == 0 || a.row_seq[r - 1] != seq;
      last = r == a.T - 1 || a.row_seq[r + 1] != seq;
      if (first && a.row_pos[r] > 0) before = a.prev + (size_t)seq * D;
    }
    const T* table_row = nullptr;
    if (EXTRA && a.table != nullptr) {
      const long long id = a.tokens[src];
      if (id >= 0 && id < a.table_rows) table_row = reinterpret_cast<const T*>(a.table) + id * a.ld_table;
    }
    const float* x_row = write_step ? a.x_in + (size_t)src * S * D : nullptr;
    float* xo_row = (a.x_out != nullptr && emit) ? a.x_out + (size_t)r * S * D : nullptr;
    const T* y_row = reinterpret_cast<const T*>(a.y) + src * a.ldy;
    const T* r_row = a.r != nullptr ? reinterpret_cast<const T*>(a.r) + src * a.ldr : nullptr;
    for (int g = g_first; g < G; g += g_step) {
      float ss = 0.f;
#pragma unroll 2
      for (int i = (sub * 32 + lane) * V; i < gs; i += wpg * 32 * V) {
        const int col = g * gs + i;
        float u[V];
#pragma unroll
        for (int v = 0; v < V; ++v) u[v] = 0.f;
        float e[V];                                     // what every stream gets besides the write step
#pragma unroll
        for (int v = 0; v < V; ++v) e[v] = 0.f;
        if (EXTRA && table_row != nullptr) {
          load_vec<T, V>(table_row + col, e);
#pragma unroll
          for (int v = 0; v < V; ++v) e[v] *= a.table_scale;
        }
        if (EXTRA && a.add != nullptr) {
          float p[V];
          load_vec<float, V>(a.add + col, p);
#pragma unroll
          for (int v = 0; v < V; ++v) e[v] += p[v];
        }
        if (write_step) {
          float x[SMAX][V], yv[V];
#pragma unroll
          for (int s = 0; s < SMAX; ++s)
            if (s < S) load_vec<float, V>(x_row + (size_t)s * D + col, x[s]);
          load_vec<T, V>(y_row + col, yv);
          if (r_row != nullptr) {
            float rv[V], bv[V];
            load_vec<T, V>(r_row + col, rv);
            load_vec<float, V>(a.rb + col, bv);
#pragma unroll
            for (int v = 0; v < V; ++v) yv[v] *= 1.f / (1.f + expf(-(rv[v] + bv[v])));
          }
#pragma unroll
          for (int t = 0; t < SMAX; ++t) {
            if (t < S) {
              float n[V];
#pragma unroll
              for (int v = 0; v < V; ++v) n[v] = fmaf(s_out[t], yv[v], e[v]);
#pragma unroll
              for (int s = 0; s < SMAX; ++s)
                if (s < S) {
#pragma unroll
                  for (int v = 0; v < V; ++v) n[v] += s_mix[s * S + t] * x[s][v];
                }
              if (xo_row != nullptr) store_vec<float, V>(xo_row + (size_t)t * D + col, n);
#pragma unroll
              for (int v = 0; v < V; ++v) u[v] += s_in[t] * n[v];
            }
          }
        } else {
          for (int t = 0; t < S; ++t) {
            if (xo_row != nullptr) store_vec<float, V>(xo_row + (size_t)t * D + col, e);
#pragma unroll
            for (int v = 0; v < V; ++v) u[v] += s_in[t] * e[v];
          }
        }
#pragma unroll
        for (int v = 0; v < V; ++v) ss += u[v] * u[v];
        store_vec<float, V>(su + col, u);
      }
      ss = warp_sum(ss);
      if (wpg > 1) {
        // one group per warp in this case, so every warp reaches the barrier once per row; two buffers take turns
        if (lane == 0) s_red[buf][warp] = ss;
        __syncthreads();
        ss = 0.f;
        for (int w = 0; w < wpg; ++w) ss += s_red[buf][g * wpg + w];
        buf ^= 1;
      }
      const float inv = 1.f / sqrtf(ss / (float)gs + a.eps);
#pragma unroll 2
      for (int i = (sub * 32 + lane) * V; i < gs; i += wpg * 32 * V) {
        const int col = g * gs + i;
        float h[V], w[V];
        load_vec<float, V>(su + col, h);
        load_vec<float, V>(a.norm_w + col, w);
#pragma unroll
        for (int v = 0; v < V; ++v) h[v] *= inv * w[v];
        if (emit) store_vec<T, V>(reinterpret_cast<T*>(a.h) + (size_t)r * a.ldh + col, h);
        if (shifted) {
          if (emit) {
            float p[V], c[V], o[V];
#pragma unroll
            for (int v = 0; v < V; ++v) p[v] = 0.f;
            if (!first) load_vec<float, V>(sprev + col, p);
            else if (before != nullptr) load_vec<float, V>(before + col, p);
            load_vec<float, V>(a.shift + col, c);
#pragma unroll
            for (int v = 0; v < V; ++v) o[v] = h[v] + (p[v] - h[v]) * c[v];
            store_vec<T, V>(reinterpret_cast<T*>(a.hs) + (size_t)r * a.ldh + col, o);
            if (last && a.state != nullptr) store_vec<float, V>(a.state + (size_t)seq * D + col, h);
          }
          store_vec<float, V>(sprev + col, h);
        }
      }
    }
    if (emit && a.ldh > D && warp == 0) {               // pad columns of the outputs stay finite
      for (int c = D + lane; c < a.ldh; c += 32) {
        reinterpret_cast<T*>(a.h)[(size_t)r * a.ldh + c] = static_cast<T>(0.f);
        if (shifted) reinterpret_cast<T*>(a.hs)[(size_t)r * a.ldh + c] = static_cast<T>(0.f);
      }
    }
  }
}

template <typename T, int S_, int V, bool EXTRA>
static int launch_stream_v(const StreamArgs& a, int blocks, int threads, size_t smem, cudaStream_t st) {
  auto kern = stream_boundary_kernel<T, S_, V, EXTRA>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return -(int)e;
  }
  kern<<<blocks, threads, smem, st>>>(a);
  return check_launch("stream_boundary_kernel");
}
template <typename T, int S_>
static int launch_stream_s(const StreamArgs& a, bool wide, int blocks, int threads, size_t smem, cudaStream_t st) {
  const bool extra = a.table != nullptr || a.add != nullptr;
  if (wide)
    return extra ? launch_stream_v<T, S_, 4, true>(a, blocks, threads, smem, st)
                 : launch_stream_v<T, S_, 4, false>(a, blocks, threads, smem, st);
  return extra ? launch_stream_v<T, S_, 1, true>(a, blocks, threads, smem, st)
               : launch_stream_v<T, S_, 1, false>(a, blocks, threads, smem, st);
}
template <typename T>
static int launch_stream(const StreamArgs& a, bool wide, int blocks, int threads, size_t smem, cudaStream_t st) {
  switch (a.S) {
    case 1: return launch_stream_s<T, 1>(a, wide, blocks, threads, smem, st);
    case 2: return launch_stream_s<T, 2>(a, wide, blocks, threads, smem, st);
    case 3: return launch_stream_s<T, 3>(a, wide, blocks, threads, smem, st);
    case 4: return launch_stream_s<T, 4>(a, wide, blocks, threads, smem, st);
    default: return launch_stream_s<T, 0>(a, wide, blocks, threads, smem, st);
  }
}

}  // namespace icb

using namespace icb;

// One sublayer boundary of the residual streams (see the head of this file). dtype is that of table, y, r, h and hs:
// bf16 or fp32; everything else is fp32. x_in == null selects the first boundary (tokens, table); with x_in, a table adds
// its rows to the streams, as add [D] (optional) does. x_out must not alias x_in. row_map and a shift exclude each
// other. rows_per_block <= 0 lets the launcher choose.
ICB_API int icb_stream_boundary(const long long* tokens, const void* table, long long ld_table, long long table_rows,
                                float table_scale, const float* add,
                                const float* x_in, float* x_out, const void* y, long long ldy, const void* r,
                                long long ldr, const float* rb, const float* mix, const float* out, const int* row_map,
                                const float* in, const float* norm_w, int groups, float eps, void* h, void* hs,
                                long long ldh, const float* shift, const float* prev, float* state, const int* row_seq,
                                const int* row_pos, int T, int S, int D, int rows_per_block, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (S < 1 || S > kMaxStreams || groups < 1 || D < 1 || D % groups || ldh < D) return -2;
  if (dtype != kBF16 && dtype != kF32) return -3;
  if (x_in == nullptr ? (tokens == nullptr || table == nullptr) : (y == nullptr || x_in == x_out)) return -4;
  if (r != nullptr && rb == nullptr) return -4;
  if (table != nullptr && tokens == nullptr) return -4;
  if (hs != nullptr && (row_map != nullptr || shift == nullptr || row_seq == nullptr || row_pos == nullptr || prev == nullptr))
    return -5;
  StreamArgs a;
  a.tokens = tokens; a.table = table; a.ld_table = ld_table; a.table_rows = table_rows; a.table_scale = table_scale; a.add = add;
  a.x_in = x_in; a.x_out = x_out; a.y = y; a.ldy = ldy; a.r = r; a.ldr = ldr; a.rb = rb; a.mix = mix; a.out = out;
  a.row_map = row_map; a.in = in; a.norm_w = norm_w; a.groups = groups; a.eps = eps;
  a.h = h; a.hs = hs; a.ldh = ldh; a.shift = shift; a.prev = prev; a.state = state;
  a.row_seq = row_seq; a.row_pos = row_pos; a.T = T; a.S = S; a.D = D;
  const int gs = D / groups;
  const bool wide = D % 4 == 0 && gs % 4 == 0 && ldh % 4 == 0 && ldy % 4 == 0 && ldr % 4 == 0 && ld_table % 4 == 0;
  // about 8 warps (16 when there are only a few rows, where latency counts): a whole number per group, but no more
  // than a group has vectors for
  const int target = T <= 2 * num_sms() ? 16 : 8;
  int warps;
  if (groups > target) {
    warps = target;                             // one group at a time per warp
  } else {
    const int lanes = wide ? (gs + 3) / 4 : gs;
    int wpg = target / groups;
    const int useful = (lanes + 31) / 32;
    if (wpg > useful) wpg = useful;
    warps = groups * wpg;
  }
  if (rows_per_block <= 0) {
    // a shifted boundary recomputes one row per block, so it wants long runs once the machine is full
    const int per_sm = 6;
    const int fill = num_sms() * per_sm;
    rows_per_block = (T + fill - 1) / fill;
    if (hs != nullptr && rows_per_block > 1 && rows_per_block < 8) rows_per_block = 8;
    if (rows_per_block > 16) rows_per_block = 16;
  }
  a.rows_per_block = rows_per_block;
  const size_t smem = (size_t)D * sizeof(float) * (hs != nullptr ? 2 : 1);
  if (smem > 200 * 1024) return -6;
  const int blocks = (T + rows_per_block - 1) / rows_per_block;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dtype == kBF16 ? launch_stream<__nv_bfloat16>(a, wide, blocks, warps * 32, smem, st)
                        : launch_stream<float>(a, wide, blocks, warps * 32, smem, st);
}
