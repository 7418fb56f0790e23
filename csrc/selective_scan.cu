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
// One more token for each of many sequences is bound by the bytes of the states: a kernel of its own, eight states per
// thread, everything straight from global memory.
#include "host_common.h"
#include "rows.cuh"

namespace icb {

constexpr int kScanThreads = 128;
constexpr int kScanTile = 16;
constexpr int kScanStep = 4;

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
  int ch_bits;              // log2 of the channels per CTA
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

// One token of NS states: S <- exp(dt A) S + du B, returns sum S C.
template <typename T, int NS>
__device__ __forceinline__ float scan_token(float dt, float du, const float (&rate)[NS], float (&s)[NS], const float* pb,
                                            const float* pc) {
  if constexpr (sizeof(T) == 4) {
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      s[i] = scan_step<T>(dt * rate[i], s[i], du * pb[i]);
      y = fmaf(s[i], pc[i], y);
    }
    return y;
  } else {
    const Pair dt2 = pair_of(dt, dt), du2 = pair_of(du, du);
    Pair y0 = pair_of(0.f, 0.f), y1 = y0;
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
      const float4 b = *reinterpret_cast<const float4*>(pb + i);
      const float4 c = *reinterpret_cast<const float4*>(pc + i);
      const float2 x0 = pair_values(pair_mul(dt2, pair_of(rate[i], rate[i + 1])));
      const float2 x1 = pair_values(pair_mul(dt2, pair_of(rate[i + 2], rate[i + 3])));
      const Pair e0 = pair_of(exp2_approx(x0.x), exp2_approx(x0.y)), e1 = pair_of(exp2_approx(x1.x), exp2_approx(x1.y));
      const Pair s0 = pair_fma(e0, pair_of(s[i], s[i + 1]), pair_mul(du2, pair_of(b.x, b.y)));
      const Pair s1 = pair_fma(e1, pair_of(s[i + 2], s[i + 3]), pair_mul(du2, pair_of(b.z, b.w)));
      y0 = pair_fma(s0, pair_of(c.x, c.y), y0);
      y1 = pair_fma(s1, pair_of(c.z, c.w), y1);
      const float2 f0 = pair_values(s0), f1 = pair_values(s1);
      s[i] = f0.x; s[i + 1] = f0.y; s[i + 2] = f1.x; s[i + 3] = f1.y;
    }
    const float2 p = pair_values(y0), q = pair_values(y1);
    return (p.x + p.y) + (q.x + q.y);
  }
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

  // two raw buffers, then the fp32 working set of the current tile; its pitch keeps the lanes of a channel, which store
  // different tokens, on different banks
  const int CP = CH + 8;
  const int raw_bytes = scan_tile_bytes<T>(CH, NB, tile);
  float* w_dt = reinterpret_cast<float*>(smem + 2 * raw_bytes);   // [tile][CP] step
  float* w_du = w_dt + tile * CP;                                 // [tile][CP] step times input
  float* w_y = w_du + tile * CP;                                  // [tile][CP]
  float* w_b = w_y + tile * CP;                                   // [tile][NW]
  float* w_c = w_b + tile * NW;                                   // [tile][NW]

  auto raw_u = [&](int buf) { return reinterpret_cast<T*>(smem + buf * raw_bytes); };
  auto raw_z = [&](int buf) { return raw_u(buf) + tile * CH; };
  auto raw_bc = [&](int buf) { return raw_z(buf) + tile * CH; };
  auto raw_dt = [&](int buf) { return reinterpret_cast<float*>(raw_bc(buf) + 2 * tile * NB); };

  auto fetch = [&](int t0, int buf) {
    const int nt = min(tile, seq.end - t0);
    const int pb = NB / V;
    const int vb = a.ch_bits - (V == 8 ? 3 : 2), fb = a.ch_bits - 2;      // pieces per row as powers of two
    for (int i = threadIdx.x; i < nt << vb; i += kScanThreads) {
      const int t = i >> vb, c = (i & ((1 << vb) - 1)) * V;
      if (c < nch) {
        cp_async16(raw_u(buf) + t * CH + c, a.u + (size_t)(t0 + t) * a.ldu + c0 + c);
        cp_async16(raw_z(buf) + t * CH + c, a.z + (size_t)(t0 + t) * a.ldz + c0 + c);
      }
    }
    for (int i = threadIdx.x; i < nt << fb; i += kScanThreads) {
      const int t = i >> fb, c = (i & ((1 << fb) - 1)) * 4;
      if (c < nch) cp_async16(raw_dt(buf) + t * CH + c, a.dt + (size_t)(t0 + t) * a.lddt + c0 + c);
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
    // whole groups of kScanStep tokens: steps of zero behind the last one, and for channels that are not there
    const int ng = (nt + kScanStep - 1) / kScanStep * kScanStep;
    {
      const int fb = a.ch_bits - 2;
      for (int i = threadIdx.x; i < ng << fb; i += kScanThreads) {
        const int t = i >> fb, ch = (i & ((1 << fb) - 1)) * 4;
        float dt[4] = {0.f, 0.f, 0.f, 0.f}, du[4] = {0.f, 0.f, 0.f, 0.f};
        if (t < nt && ch < nch) {
          float raw[4], bias[4];
          load_f32<4>(raw_dt(buf) + t * CH + ch, raw);
          load_f32<4>(a.dt_bias + c0 + ch, bias);
          const T* u = raw_u(buf) + t * CH + ch;
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            dt[e] = softplus_of<T>(raw[e] + bias[e]);
            du[e] = dt[e] * static_cast<float>(u[e]);
          }
        }
        store_f32<4>(w_dt + t * CP + ch, dt);
        store_f32<4>(w_du + t * CP + ch, du);
      }
    }
    for (int i = threadIdx.x; i < ng * NW; i += kScanThreads) {
      const int t = i / NW, n = i - t * NW;
      const bool on = t < nt && n < a.N;
      w_b[i] = on ? static_cast<float>(raw_bc(buf)[t * NB + n]) : 0.f;
      w_c[i] = on ? static_cast<float>(raw_bc(buf)[(tile + t) * NB + n]) : 0.f;
    }
    __syncthreads();
    // kScanStep tokens at a time: their loads are in flight together, and their sums over the channel's lanes are shared out
    // so that a lane ends up with some of the tokens
    for (int t0s = 0; t0s < ng; t0s += kScanStep) {
      float y[kScanStep];
#pragma unroll
      for (int q = 0; q < kScanStep; ++q) {
        const int t = t0s + q;
        const float dt = w_dt[t * CP + my], du = w_du[t * CP + my];
        y[q] = scan_token<T, NS>(dt, du, a2, s, w_b + t * NW + n0, w_c + t * NW + n0);
      }
      int off = 1, first = 0, mine = kScanStep;              // this lane's tokens: first .. first + mine
#pragma unroll
      for (int half = kScanStep / 2; half > 0; half >>= 1) {
        if (off >= a.lanes) break;
        const bool up = sub & off;
#pragma unroll
        for (int i = 0; i < half; ++i) {
          const float keep = up ? y[half + i] : y[i], give = up ? y[i] : y[half + i];
          y[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
        }
        first += up ? half : 0;
        mine = half;
        off <<= 1;
      }
      for (int o = off; o < a.lanes; o <<= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], o);
      if (sub < off) {
#pragma unroll
        for (int i = 0; i < kScanStep; ++i)
          if (i < mine) w_y[(t0s + first + i) * CP + my] = y[i];
      }
    }
    __syncthreads();
    const int vb = a.ch_bits - (V == 8 ? 3 : 2);
    for (int i = threadIdx.x; i < nt << vb; i += kScanThreads) {
      const int t = i >> vb, ch = (i & ((1 << vb) - 1)) * V;
      if (ch >= nch) continue;
      float u[V], z[V], d[V], y[V];
      load_row<T>(raw_u(buf) + t * CH + ch, u);
      load_row<T>(raw_z(buf) + t * CH + ch, z);
      load_f32<V>(a.d + c0 + ch, d);
      load_f32<V>(w_y + t * CP + ch, y);
#pragma unroll
      for (int v = 0; v < V; ++v) y[v] = fmaf(d[v], u[v], y[v]) * silu_of<T>(z[v]);
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

template <typename T>
__device__ __forceinline__ void load_four(const T* p, float (&f)[4]) {
  if constexpr (sizeof(T) == 4) {
    load_f32<4>(p, f);
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  }
}

constexpr int kScanOneThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kScanOneThreads, 5) scan_one_kernel(const ScanArgs<T> a) {
  constexpr int Q = 2;                                 // quads of states per lane, their loads in flight together
  const int idx = blockIdx.x * kScanOneThreads + threadIdx.x;
  const int sub = idx & (a.lanes - 1), c = idx >> a.ch_bits, r = blockIdx.y;      // ch_bits: log2 of the lanes here
  const bool live = c < a.C;
  float y = 0.f, u = 0.f, z = 0.f, d = 0.f;
  if (live) {
    float* st = a.state + ((size_t)a.seqs[r] * a.C + c) * a.NP;
    const bool fresh = a.pos[r] == 0;
    const T* bc = a.bc + (size_t)r * a.ldbc;
    u = static_cast<float>(a.u[(size_t)r * a.ldu + c]);
    z = static_cast<float>(a.z[(size_t)r * a.ldz + c]);
    d = a.d[c];
    const float raw = a.dt[(size_t)r * a.lddt + c] + a.dt_bias[c];
    float dt = 0.f, du = 0.f;
    for (int base = sub * 4 * Q; base < a.NP; base += a.lanes * 4 * Q) {
      float4 s4[Q];
      float rate[Q][4], b[Q][4], k[Q][4];
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int n0 = base + q * 4;
        s4[q] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (n0 >= a.NP) continue;
        if (!fresh) s4[q] = *reinterpret_cast<const float4*>(st + n0);
        load_f32<4>(a.a_log + (size_t)c * a.NP + n0, rate[q]);
        load_four<T>(bc + a.b_col + n0, b[q]);
        load_four<T>(bc + a.c_col + n0, k[q]);
      }
      if (base < a.lanes * 4 * Q) {
        dt = softplus_of<T>(raw);
        du = dt * u;
      }
#pragma unroll
      for (int q = 0; q < Q; ++q) {
        const int n0 = base + q * 4;
        if (n0 >= a.NP) continue;
        float s[4] = {s4[q].x, s4[q].y, s4[q].z, s4[q].w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          if (n0 + e < a.N) {
            const float x = sizeof(T) == 4 ? -expf(rate[q][e]) : __expf(rate[q][e]) * -1.4426950408889634f;
            s[e] = scan_step<T>(dt * x, s[e], du * b[q][e]);
            y = fmaf(s[e], k[q][e], y);
          } else {
            s[e] = 0.f;
          }
        }
        *reinterpret_cast<float4*>(st + n0) = make_float4(s[0], s[1], s[2], s[3]);
      }
    }
  }
  for (int o = a.lanes >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (live && sub == 0) a.y[(size_t)r * a.ldy + c] = static_cast<T>(fmaf(d, u, y) * silu_of<T>(z));
}

template <typename T>
static int launch_scan_one(ScanArgs<T> a, int rows, cudaStream_t st) {
  a.ch_bits = 0;
  while (a.ch_bits < 5 && 8 << a.ch_bits < a.NP) ++a.ch_bits;
  a.lanes = 1 << a.ch_bits;
  dim3 grid((int)(((long long)a.C * a.lanes + kScanOneThreads - 1) / kScanOneThreads), rows);
  scan_one_kernel<T><<<grid, kScanOneThreads, 0, st>>>(a);
  return check_launch("scan_one_kernel");
}

template <typename T, int NS>
static int launch_scan_ns(ScanArgs<T> a, int sequences, int longest, cudaStream_t st) {
  int lanes = 1;
  while (lanes * NS < a.N) lanes *= 2;
  if (lanes > 16) return -6;
  a.lanes = lanes;
  const int ch = kScanThreads / lanes, nb = (a.N + kVec<T> - 1) / kVec<T> * kVec<T>, nw = lanes * NS;
  int tile = (longest + kScanStep - 1) / kScanStep * kScanStep;
  if (tile > kScanTile) tile = kScanTile;
  a.ch_bits = 0;
  while (1 << a.ch_bits < ch) ++a.ch_bits;
  const size_t smem = 2 * (size_t)scan_tile_bytes<T>(ch, nb, tile) + (size_t)tile * (3 * (ch + 8) + 2 * nw) * 4;
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
  if (a.cu == nullptr) return launch_scan_one<T>(a, sequences, st);
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
// states per lane (4, 8, 12, 16 or 32; N <= 16 per_lane; unused without cu). C and all pitches are multiples of 8, b_col and c_col too, NP
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
                  (T*)y, ldy, seqs, pos, cu, C, N, NP, 0, 0};
    return launch_scan<T>(a, sequences, longest, per_lane, st);
  }
  if (dtype == kF32) {
    ScanArgs<float> a{(const float*)u, dt, (const float*)z, (const float*)bc, ldu, lddt, ldz, ldbc, b_col, c_col, dt_bias,
                      a_log, d, state, (float*)y, ldy, seqs, pos, cu, C, N, NP, 0, 0};
    return launch_scan<float>(a, sequences, longest, per_lane, st);
  }
  return -3;
}
