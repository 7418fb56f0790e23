// Selective scan with a diagonal state per channel (fp32, carried from batch to batch for every sequence):
//
//   dt = softplus(raw + bias)          S[n] <- exp(dt A[n]) S[n] + dt u B[n]          y = (sum_n S[n] C[n] + D u) silu(z)
//
// A CTA owns a block of channels of one sequence and walks its rows in tiles of kScanTile. A tile's u, raw step, z, B
// and C rows arrive by asynchronous copies while the tile before is computed. What depends on one element only
// (softplus, dt u on the way in; D u, silu and the conversion on the way out) is done once per element by all threads;
// the loop over time in between touches shared memory and registers alone. A channel's states are spread over
// `lanes` neighbouring lanes with NS each. In 16-bit models exp runs in the base-2 domain with log2(e) folded into A; in
// fp32 models a state that hardly decays would add up that function's error over thousands of tokens, so there
// S <- S + (expm1(dt A) S + dt u B).
// Decoding is the same kernel with one row per sequence and wider channel blocks.
#include "host_common.h"
#include "rows.cuh"

namespace icb {

constexpr int kScanThreads = 128;
constexpr int kScanTile = 16;

template <typename T>
struct ScanArgs {
  const T* u;               // [rows, ldu] convolved input
  const float* dt;          // [rows, lddt] raw step
  const T* z;               // [rows, ldz] gate
  const T* bc;              // [rows, ldbc]: B at b_col, C at c_col
  long long ldu, lddt, ldz, ldbc;
  int b_col, c_col;
  const float* dt_bias;     // [C]
  const float* a_log;       // [C, NP], A = -exp(a_log)
  const float* d;           // [C]
  float* state;             // [slots, C, NP]
  T* y;                     // [rows, ldy]
  long long ldy;
  const int* seqs;
  const int* pos;
  const int* cu;            // [sequences + 1] or null: one row each
  int C, N, NP;             // channels (multiple of 8), states, their pitch (multiple of 4)
  int lanes;                // lanes per channel, a power of two up to 16
};

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <typename T>
__device__ __forceinline__ float scan_step(float x, float s, float in) {
  if constexpr (sizeof(T) == 4) return s + fmaf(expm1f(x), s, in);
  return fmaf(exp2_approx(x), s, in);
}

// Shared memory of one tile buffer, in bytes; CH channels, NB = lanes * NS padded states.
template <typename T>
__host__ __device__ inline int scan_tile_bytes(int ch, int nb, int tile) {
  return tile * (ch * (2 * (int)sizeof(T) + 4) + 2 * nb * (int)sizeof(T));
}

template <typename T, int NS>
__global__ void __launch_bounds__(kScanThreads) selective_scan_kernel(const ScanArgs<T> a, int tile) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int V = kVec<T>;
  const int CH = kScanThreads / a.lanes;
  const int c0 = blockIdx.x * CH;
  const int nch = min(CH, a.C - c0);                    // multiple of 8
  const int NB = (a.N + V - 1) / V * V;                 // copied states per token (16-byte pieces)
  const int NW = a.lanes * NS;                          // states that the lanes of a channel read
  const SeqRows seq = seq_rows(a.cu, a.seqs, a.pos, blockIdx.y);
  if (seq.begin >= seq.end) return;

  // two raw buffers, then the fp32 working set of the current tile
  const int raw_bytes = scan_tile_bytes<T>(CH, NB, tile);
  float* w_dt = reinterpret_cast<float*>(smem + 2 * raw_bytes);   // [tile][CH] step
  float* w_du = w_dt + tile * CH;                                 // [tile][CH] step times input
  float* w_y = w_du + tile * CH;                                  // [tile][CH]
  float* w_b = w_y + tile * CH;                                   // [tile][NW]
  float* w_c = w_b + tile * NW;                                   // [tile][NW]

  auto raw_u = [&](int buf) { return reinterpret_cast<T*>(smem + buf * raw_bytes); };
  auto raw_z = [&](int buf) { return raw_u(buf) + tile * CH; };
  auto raw_bc = [&](int buf) { return raw_z(buf) + tile * CH; };
  auto raw_dt = [&](int buf) { return reinterpret_cast<float*>(raw_bc(buf) + 2 * tile * NB); };

  auto fetch = [&](int t0, int buf) {
    const int nt = min(tile, seq.end - t0);
    const int pv = nch / V, pf = nch / 4, pb = NB / V;
    for (int i = threadIdx.x; i < nt * pv; i += kScanThreads) {
      const int t = i / pv, c = (i - t * pv) * V;
      cp_async16(raw_u(buf) + t * CH + c, a.u + (size_t)(t0 + t) * a.ldu + c0 + c);
      cp_async16(raw_z(buf) + t * CH + c, a.z + (size_t)(t0 + t) * a.ldz + c0 + c);
    }
    for (int i = threadIdx.x; i < nt * pf; i += kScanThreads) {
      const int t = i / pf, c = (i - t * pf) * 4;
      cp_async16(raw_dt(buf) + t * CH + c, a.dt + (size_t)(t0 + t) * a.lddt + c0 + c);
    }
    for (int i = threadIdx.x; i < nt * pb; i += kScanThreads) {
      const int t = i / pb, c = (i - t * pb) * V;
      const T* row = a.bc + (size_t)(t0 + t) * a.ldbc;
      cp_async16(raw_bc(buf) + t * NB + c, row + a.b_col + c);
      cp_async16(raw_bc(buf) + (tile + t) * NB + c, row + a.c_col + c);
    }
    cp_async_commit();
  };

  fetch(seq.begin, 0);

  const int my = threadIdx.x / a.lanes, sub = threadIdx.x - my * a.lanes;
  const int c = c0 + my;
  const bool live = my < nch;
  const int n0 = sub * NS;
  float s[NS], a2[NS];
#pragma unroll
  for (int i = 0; i < NS; ++i) { s[i] = 0.f; a2[i] = 0.f; }
  float* st = a.state + ((size_t)seq.slot * a.C + c) * a.NP + n0;
  if (live) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
      if (n0 + i < a.NP) {
        const float4 al = *reinterpret_cast<const float4*>(a.a_log + (size_t)c * a.NP + n0 + i);
        const float l[4] = {al.x, al.y, al.z, al.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
          if (n0 + i + e < a.N) a2[i + e] = sizeof(T) == 4 ? -expf(l[e]) : -expf(l[e]) * 1.4426950408889634f;
        if (!seq.fresh) {
          const float4 u = *reinterpret_cast<const float4*>(st + i);
          s[i] = u.x; s[i + 1] = u.y; s[i + 2] = u.z; s[i + 3] = u.w;
        }
      }
    }
  }

  int buf = 0;
  for (int t0 = seq.begin; t0 < seq.end; t0 += tile, buf ^= 1) {
    const int nt = min(tile, seq.end - t0);
    const bool more = t0 + tile < seq.end;
    if (more) {
      fetch(t0 + tile, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * nch; i += kScanThreads) {
      const int t = i / nch, ch = i - t * nch, k = t * CH + ch;
      const float dt = softplus_f32(raw_dt(buf)[k] + a.dt_bias[c0 + ch]);
      w_dt[k] = dt;
      w_du[k] = dt * static_cast<float>(raw_u(buf)[k]);
    }
    for (int i = threadIdx.x; i < nt * NW; i += kScanThreads) {
      const int t = i / NW, n = i - t * NW;
      w_b[i] = n < a.N ? static_cast<float>(raw_bc(buf)[t * NB + n]) : 0.f;
      w_c[i] = n < a.N ? static_cast<float>(raw_bc(buf)[(tile + t) * NB + n]) : 0.f;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float dt = live ? w_dt[t * CH + my] : 0.f;
      const float du = live ? w_du[t * CH + my] : 0.f;
      const float* pb = w_b + t * NW + n0;
      const float* pc = w_c + t * NW + n0;
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int i = 0; i < NS; i += 4) {
        const float4 b = *reinterpret_cast<const float4*>(pb + i);
        const float4 k = *reinterpret_cast<const float4*>(pc + i);
        s[i] = scan_step<T>(dt * a2[i], s[i], du * b.x);
        s[i + 1] = scan_step<T>(dt * a2[i + 1], s[i + 1], du * b.y);
        s[i + 2] = scan_step<T>(dt * a2[i + 2], s[i + 2], du * b.z);
        s[i + 3] = scan_step<T>(dt * a2[i + 3], s[i + 3], du * b.w);
        y0 = fmaf(s[i], k.x, y0);
        y1 = fmaf(s[i + 1], k.y, y1);
        y0 = fmaf(s[i + 2], k.z, y0);
        y1 = fmaf(s[i + 3], k.w, y1);
      }
      float y = y0 + y1;
      for (int o = a.lanes >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (sub == 0) w_y[t * CH + my] = y;
    }
    __syncthreads();
    const int pv = nch / V;
    for (int i = threadIdx.x; i < nt * pv; i += kScanThreads) {
      const int t = i / pv, ch = (i - t * pv) * V;
      float u[V], z[V], d[V], y[V];
      load_row<T>(raw_u(buf) + t * CH + ch, u);
      load_row<T>(raw_z(buf) + t * CH + ch, z);
      load_f32<V>(a.d + c0 + ch, d);
      load_f32<V>(w_y + t * CH + ch, y);
#pragma unroll
      for (int v = 0; v < V; ++v) y[v] = fmaf(d[v], u[v], y[v]) * silu_f32(z[v]);
      store_row<T>(a.y + (size_t)(t0 + t) * a.ldy + c0 + ch, y);
    }
    if (more) __syncthreads();       // the buffer read here is the one that the next fetch fills
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < NS; i += 4)
      if (n0 + i < a.NP) *reinterpret_cast<float4*>(st + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
  }
}

template <typename T, int NS>
static int launch_scan_ns(ScanArgs<T> a, int sequences, int longest, cudaStream_t st) {
  int lanes = 1;
  while (lanes * NS < a.N) lanes *= 2;
  if (lanes > 16) return -6;
  a.lanes = lanes;
  const int ch = kScanThreads / lanes, nb = (a.N + kVec<T> - 1) / kVec<T> * kVec<T>, nw = lanes * NS;
  const int tile = longest < kScanTile ? longest : kScanTile;
  const size_t smem = 2 * (size_t)scan_tile_bytes<T>(ch, nb, tile) + (size_t)tile * (3 * ch + 2 * nw) * 4;
  auto kern = selective_scan_kernel<T, NS>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return -(int)e;
  }
  dim3 grid((a.C + ch - 1) / ch, sequences);
  kern<<<grid, kScanThreads, smem, st>>>(a, tile);
  return check_launch("selective_scan_kernel");
}

template <typename T>
static int launch_scan(const ScanArgs<T>& a, int sequences, int longest, int ns, cudaStream_t st) {
  switch (ns) {
    case 4: return launch_scan_ns<T, 4>(a, sequences, longest, st);
    case 8: return launch_scan_ns<T, 8>(a, sequences, longest, st);
    case 12: return launch_scan_ns<T, 12>(a, sequences, longest, st);
    case 16: return launch_scan_ns<T, 16>(a, sequences, longest, st);
    case 32: return launch_scan_ns<T, 32>(a, sequences, longest, st);
    default: return -5;
  }
}

}  // namespace icb

using namespace icb;

// Selective scan of rows of `sequences` sequences (cu [sequences + 1]; null: one row each, sequences = rows). dtype is
// that of u, z, bc and y (bf16 or fp32); everything else is fp32. `longest` bounds the rows of one sequence. `per_lane`
// states per lane (4, 8, 12, 16 or 32; N <= 16 per_lane). C and all pitches are multiples of 8, b_col and c_col too, NP
// is N rounded up to 4, and rows of bc are readable up to N rounded up to 8 columns behind b_col and c_col.
ICB_API int icb_selective_scan(const void* u, long long ldu, const float* dt, long long lddt, const void* z, long long ldz,
                               const void* bc, long long ldbc, int b_col, int c_col, const float* dt_bias,
                               const float* a_log, const float* d, float* state, void* y, long long ldy, const int* seqs,
                               const int* pos, const int* cu, int sequences, int longest, int C, int N, int per_lane,
                               int dtype, void* stream) {
  if (sequences <= 0 || C <= 0) return 0;
  if (sequences > 65535) return -2;
  if (C % 8 || ldu % 8 || lddt % 8 || ldz % 8 || ldbc % 8 || ldy % 8 || b_col % 8 || c_col % 8) return -2;
  if (N < 1 || longest < 1 || (cu == nullptr && longest != 1)) return -4;
  const int NP = (N + 3) / 4 * 4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16) {
    using T = __nv_bfloat16;
    ScanArgs<T> a{(const T*)u, dt, (const T*)z, (const T*)bc, ldu, lddt, ldz, ldbc, b_col, c_col, dt_bias, a_log, d, state,
                  (T*)y, ldy, seqs, pos, cu, C, N, NP, 0};
    return launch_scan<T>(a, sequences, longest, per_lane, st);
  }
  if (dtype == kF32) {
    ScanArgs<float> a{(const float*)u, dt, (const float*)z, (const float*)bc, ldu, lddt, ldz, ldbc, b_col, c_col, dt_bias,
                      a_log, d, state, (float*)y, ldy, seqs, pos, cu, C, N, NP, 0};
    return launch_scan<float>(a, sequences, longest, per_lane, st);
  }
  return -3;
}
