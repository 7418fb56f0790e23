// Gated delta rule with a decay per key channel, fp32 state [dim x vdim] per head carried from batch to batch:
//
//   S <- g S          u = beta (v - S^T k)          S <- S + k u^T          o = S^T q
//
// Three kernels, each for any mixture of sequences (rows.cuh):
//   delta_prepare   short convolution + silu of q, k and v, unit norms of q and k, q . k, decay factors, beta
//   delta_rule      the recurrence
//   delta_output    RMS norm of a head's output, gain, output gate
//
// delta_rule: the columns of S do not depend on one another, so a warp owns 16 of them (four per group of eight lanes,
// the key channels spread over the eight lanes, 4 columns x DIM / 8 channels in a thread's registers). With
// S' = g S both products of a step, S'^T k and S'^T q, come out of one pass over the registers; o = S'^T q + u (k . q).
// The eight lanes' partial sums meet in a transposing reduction (seven shuffles for eight values). k, q, g and v rows of
// the next tile of tokens arrive by asynchronous copies meanwhile.
#include "host_common.h"
#include "rows.cuh"

namespace icb {

template <typename T>
struct DeltaPrepArgs {
  ConvArgs<T> conv;            // channels [q: G x K | k: G x K | v: H x V]
  const T* beta_in;            // [rows, ldbeta] H logits
  long long ldbeta;
  float* a;                    // [rows, H x K] decay input, replaced by the decay factor
  const float* a_log;          // [H]
  const float* dt_bias;        // [H x K]
  float* q;                    // [rows, G x K] unit vectors times q_scale
  float* k;                    // [rows, G x K]
  float* qk;                   // [rows, G] their products
  T* v;                        // [rows, H x V]
  float* beta;                 // [rows, H]
  int rows, G, H, K, V;        // K, V: multiples of 8
  float q_scale;
  int run, keep, lanes;        // lanes of a q / k head: a power of two
};

constexpr float kUnitEps = 1e-6f;

template <typename T, int TAPS>
__global__ void __launch_bounds__(128) delta_prepare_kernel(const DeltaPrepArgs<T> p) {
  constexpr int W = kVec<T>;
  constexpr int S = sizeof(T) == 4 ? 2 : 1;           // pieces of a q / k head that one lane holds
  const ConvArgs<T>& a = p.conv;
  const int r0 = blockIdx.x * p.run, r1 = min(p.rows, r0 + p.run);
  if (r0 >= p.rows) return;
  // thread roles, each rounded up to whole warps: q / k heads, v channels, decay channels, beta
  int task = blockIdx.y * blockDim.x + threadIdx.x;
  const int n_qk = (p.G * p.lanes + 31) & ~31, n_v = (p.H * p.V / W + 31) & ~31, n_g = (p.H * p.K / 4 + 31) & ~31;
  const int most = (TAPS > 0 ? TAPS : a.taps) - 1;
  if (task < n_qk + n_v) {
    const bool is_v = task >= n_qk;
    if (is_v) task -= n_qk;
    const int head = is_v ? 0 : task / p.lanes, sub = is_v ? 0 : task - head * p.lanes;
    bool live[S];
    int ch[S];
    ConvWeights<T, TAPS> wq[S], wk[S];
#pragma unroll
    for (int e = 0; e < S; ++e) {
      const int c = (sub + e * p.lanes) * W;
      live[e] = is_v ? e == 0 && task < p.H * p.V / W : head < p.G && c < p.K;
      ch[e] = is_v ? 2 * p.G * p.K + task * W : head * p.K + c;
      if (live[e]) {
        load_conv_weights<T, TAPS>(a, ch[e], wq[e]);
        if (!is_v) load_conv_weights<T, TAPS>(a, p.G * p.K + ch[e], wk[e]);
      }
    }
    int before = rows_before(a.seqs, r0, most), slot = a.seqs[r0];
    for (int r = r0; r < r1; ++r) {
      if (r > r0) {
        const int s = a.seqs[r];
        before = s == slot ? min(before + 1, most) : 0;
        slot = s;
      }
      const int pos = a.pos[r];
      float x[S][W], y[S][W];
      if (is_v) {
        if (live[0]) {
          conv_silu_row<T, TAPS>(a, wq[0], r, before, slot, pos, ch[0], x[0]);
          store_row<T>(p.v + (size_t)r * p.H * p.V + task * W, x[0]);
          if (p.keep) conv_keep<T>(a, r, before, slot, pos, ch[0]);
        }
        continue;
      }
      float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
      for (int e = 0; e < S; ++e) {
        if (!live[e]) continue;
        conv_silu_row<T, TAPS>(a, wq[e], r, before, slot, pos, ch[e], x[e]);
        conv_silu_row<T, TAPS>(a, wk[e], r, before, slot, pos, p.G * p.K + ch[e], y[e]);
#pragma unroll
        for (int i = 0; i < W; ++i) {
          qq = fmaf(x[e][i], x[e][i], qq);
          kk = fmaf(y[e][i], y[e][i], kk);
          qk = fmaf(x[e][i], y[e][i], qk);
        }
      }
      for (int o = p.lanes >> 1; o > 0; o >>= 1) {
        qq += __shfl_xor_sync(0xffffffffu, qq, o);
        kk += __shfl_xor_sync(0xffffffffu, kk, o);
        qk += __shfl_xor_sync(0xffffffffu, qk, o);
      }
      const float fq = p.q_scale / sqrtf(qq + kUnitEps), fk = 1.f / sqrtf(kk + kUnitEps);
#pragma unroll
      for (int e = 0; e < S; ++e) {
        if (!live[e]) continue;
#pragma unroll
        for (int i = 0; i < W; ++i) { x[e][i] *= fq; y[e][i] *= fk; }
        store_f32<W>(p.q + (size_t)r * p.G * p.K + ch[e], x[e]);
        store_f32<W>(p.k + (size_t)r * p.G * p.K + ch[e], y[e]);
        if (e == 0 && sub == 0) p.qk[(size_t)r * p.G + head] = qk * fq * fk;
        if (p.keep) {
          conv_keep<T>(a, r, before, slot, pos, ch[e]);
          conv_keep<T>(a, r, before, slot, pos, p.G * p.K + ch[e]);
        }
      }
    }
    return;
  }
  task -= n_qk + n_v;
  if (task < n_g) {
    if (task >= p.H * p.K / 4) return;
    const int ch = task * 4;
    const float rate = -expf(p.a_log[ch / p.K]);
    float bias[4];
    load_f32<4>(p.dt_bias + ch, bias);
    for (int r = r0; r < r1; ++r) {
      float* at = p.a + (size_t)r * p.H * p.K + ch;
      float f[4];
      load_f32<4>(at, f);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float x = rate * softplus_f32(f[i] + bias[i]);
        // factors near one act thousands of times: in fp32 models they are rounded once
        f[i] = sizeof(T) == 4 ? (float)exp((double)x) : expf(x);
      }
      store_f32<4>(at, f);
    }
    return;
  }
  task -= n_g;
  if (task >= p.H) return;
  for (int r = r0; r < r1; ++r)
    p.beta[(size_t)r * p.H + task] = sigmoid_f32(static_cast<float>(p.beta_in[(size_t)r * p.ldbeta + task]));
}

// ---------------------------------------------------------------------------------------------------------
constexpr int kDeltaTile = 8;         // tokens per shared-memory buffer

template <typename T>
struct DeltaArgs {
  const float* q;              // [rows, G x K]
  const float* k;
  const float* g;              // [rows, H x K]
  const float* qk;             // [rows, G]
  const T* v;                  // [rows, H x V]
  const float* beta;           // [rows, H]
  float* state;                // [slots, H, V, KP], KP = K rounded up to 32
  float* o;                    // [rows, H x V]
  const int* seqs;
  const int* pos;
  const int* cu;
  int G, H, K, V;
};

template <typename T, int NJ>         // NJ * 32 >= K
__global__ void __launch_bounds__(128) delta_rule_kernel(const DeltaArgs<T> a, int tile) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr int KP = NJ * 32;
  const SeqRows seq = seq_rows(a.cu, a.seqs, a.pos, blockIdx.x);
  if (seq.begin >= seq.end) return;
  const int h = blockIdx.y, kvh = h / (a.H / a.G);
  const int warps = blockDim.x >> 5, cols = warps * 16;          // columns of this CTA
  const int col_base = blockIdx.z * cols, ncol = min(cols, a.V - col_base);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane & 7;
  const int lc = warp * 16 + (lane >> 3) * 4;                    // first of this thread's four columns inside the CTA
  const int col = col_base + lc;
  const bool live = lc < ncol;                                   // V is a multiple of 4: all four or none

  // per buffer: k, q, g [tile][KP] fp32, v [tile][cols] T, beta and qk [tile] fp32
  const int buf_bytes = tile * (3 * KP * 4 + cols * (int)sizeof(T)) + ((tile * 8 + 15) & ~15);
  auto vec = [&](int buf, int which) { return reinterpret_cast<float*>(smem + buf * buf_bytes) + which * tile * KP; };
  auto vbuf = [&](int buf) { return reinterpret_cast<T*>(smem + buf * buf_bytes + tile * 3 * KP * 4); };
  auto sbuf = [&](int buf) { return reinterpret_cast<float*>(smem + buf * buf_bytes + tile * (3 * KP * 4 + cols * (int)sizeof(T))); };

  auto fetch = [&](int t0, int buf) {
    const int nt = min(tile, seq.end - t0);
    const int pk = a.K / 4;
    for (int i = threadIdx.x; i < nt * pk; i += blockDim.x) {
      const int t = i / pk, c = (i - t * pk) * 4;
      const size_t row = (size_t)(t0 + t);
      cp_async16(vec(buf, 0) + t * KP + c, a.k + (row * a.G + kvh) * a.K + c);
      cp_async16(vec(buf, 1) + t * KP + c, a.q + (row * a.G + kvh) * a.K + c);
      cp_async16(vec(buf, 2) + t * KP + c, a.g + (row * a.H + h) * a.K + c);
    }
    const int pv = ncol / kVec<T>;
    for (int i = threadIdx.x; i < nt * pv; i += blockDim.x) {
      const int t = i / pv, c = (i - t * pv) * kVec<T>;
      cp_async16(vbuf(buf) + t * cols + c, a.v + ((size_t)(t0 + t) * a.H + h) * a.V + col_base + c);
    }
    cp_async_commit();
    for (int t = threadIdx.x; t < nt; t += blockDim.x) {
      sbuf(buf)[t] = a.beta[(size_t)(t0 + t) * a.H + h];
      sbuf(buf)[tile + t] = a.qk[(size_t)(t0 + t) * a.G + kvh];
    }
  };

  if (KP > a.K) {        // pad channels hold zeros in both buffers and stay so: the copies do not touch them
    const int pad = KP - a.K;
    for (int i = threadIdx.x; i < 2 * 3 * tile * pad; i += blockDim.x) {
      const int b = i / (3 * tile * pad), rest = i - b * (3 * tile * pad);
      vec(b, 0)[(rest / pad) * KP + a.K + rest % pad] = 0.f;
    }
  }
  fetch(seq.begin, 0);

  float s[4][NJ][4];
  float* st = a.state + (((size_t)seq.slot * a.H + h) * a.V + col) * KP + kl * 4;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !seq.fresh) u = *reinterpret_cast<const float4*>(st + (size_t)c * KP + j * 32);
      s[c][j][0] = u.x; s[c][j][1] = u.y; s[c][j][2] = u.z; s[c][j][3] = u.w;
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
    const float* pk = vec(buf, 0) + kl * 4;
    const float* pq = vec(buf, 1) + kl * 4;
    const float* pg = vec(buf, 2) + kl * 4;
    for (int t = 0; t < nt; ++t) {
      float sum[8];                       // S'^T k of the four columns, then S'^T q
#pragma unroll
      for (int i = 0; i < 8; ++i) sum[i] = 0.f;
      float4 kk[NJ];
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        kk[j] = *reinterpret_cast<const float4*>(pk + t * KP + j * 32);
        const float4 qq = *reinterpret_cast<const float4*>(pq + t * KP + j * 32);
        const float4 gg = *reinterpret_cast<const float4*>(pg + t * KP + j * 32);
        const float kf[4] = {kk[j].x, kk[j].y, kk[j].z, kk[j].w}, qf[4] = {qq.x, qq.y, qq.z, qq.w},
                    gf[4] = {gg.x, gg.y, gg.z, gg.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            s[c][j][i] *= gf[i];
            sum[c] = fmaf(s[c][j][i], kf[i], sum[c]);
            sum[4 + c] = fmaf(s[c][j][i], qf[i], sum[4 + c]);
          }
      }
      // eight sums over eight lanes: lane kl ends up with the total of sum[kl]
      const bool hi4 = kl & 4, hi2 = kl & 2, hi1 = kl & 1;
      float r4[4], r2[2], tot;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float keep = hi4 ? sum[4 + i] : sum[i], give = hi4 ? sum[i] : sum[4 + i];
        r4[i] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float keep = hi2 ? r4[2 + i] : r4[i], give = hi2 ? r4[i] : r4[2 + i];
        r2[i] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
      }
      {
        const float keep = hi1 ? r2[1] : r2[0], give = hi1 ? r2[0] : r2[1];
        tot = keep + __shfl_xor_sync(0xffffffffu, give, 1);
      }
      const float beta = sbuf(buf)[t], qk = sbuf(buf)[tile + t];
      const float vv = live ? static_cast<float>(vbuf(buf)[t * cols + lc + (kl & 3)]) : 0.f;
      const float mine = beta * (vv - tot);             // meaningful on lanes 0..3 of the group
      float u[4];
#pragma unroll
      for (int c = 0; c < 4; ++c) u[c] = __shfl_sync(0xffffffffu, mine, c, 8);
      if (hi4 && live) {
        const float uc = hi2 ? (hi1 ? u[3] : u[2]) : (hi1 ? u[1] : u[0]);
        a.o[((size_t)(t0 + t) * a.H + h) * a.V + col + (kl & 3)] = fmaf(uc, qk, tot);
      }
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const float kf[4] = {kk[j].x, kk[j].y, kk[j].z, kk[j].w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int c = 0; c < 4; ++c) s[c][j][i] = fmaf(kf[i], u[c], s[c][j][i]);
      }
    }
    if (more) __syncthreads();            // this buffer is the next but one fetch's target
  }
  if (live) {
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < NJ; ++j)
        *reinterpret_cast<float4*>(st + (size_t)c * KP + j * 32) = make_float4(s[c][j][0], s[c][j][1], s[c][j][2], s[c][j][3]);
  }
}

template <typename T, int NJ>
static int launch_delta(const DeltaArgs<T>& a, int sequences, int longest, cudaStream_t st) {
  // 64 columns per CTA unless that leaves SMs without one
  int warps = 4;
  while (warps > 1 && (warps * 16 >= 2 * a.V || (long long)sequences * a.H * ((a.V + warps * 16 - 1) / (warps * 16)) < 2 * num_sms()))
    warps >>= 1;
  const int cols = warps * 16, tile = longest < kDeltaTile ? longest : kDeltaTile;
  const size_t smem = 2 * (size_t)(tile * (3 * NJ * 32 * 4 + cols * (int)sizeof(T)) + ((tile * 8 + 15) & ~15));
  auto kern = delta_rule_kernel<T, NJ>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return -(int)e;
  }
  dim3 grid(sequences, a.H, (a.V + cols - 1) / cols);
  kern<<<grid, warps * 32, smem, st>>>(a, tile);
  return check_launch("delta_rule_kernel");
}

// ---------------------------------------------------------------------------------------------------------
// y[r, head] = o / rms(o over the head's `valid` values) * w * sigmoid(gate) * scale, one head per group of lanes
template <typename T>
__global__ void __launch_bounds__(256) delta_output_kernel(const float* __restrict__ o, const float* __restrict__ gate,
                                                           long long ldg, const float* __restrict__ w, float eps,
                                                           float scale, T* __restrict__ y, long long ldy, int rows, int H,
                                                           int V, int valid, int lanes) {
  constexpr int W = kVec<T>;
  const long long unit = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / lanes;
  const int sub = threadIdx.x % lanes;
  const bool live = unit < (long long)rows * H;
  const int r = live ? (int)(unit / H) : 0, h = live ? (int)(unit - (long long)r * H) : 0;
  const float* src = o + ((size_t)r * H + h) * V;
  float ss = 0.f;
  if (live)
    for (int c = sub * W; c < V; c += lanes * W) {
      float f[W];
      load_f32<W>(src + c, f);
#pragma unroll
      for (int i = 0; i < W; ++i) ss = fmaf(f[i], f[i], ss);      // the padding holds zeros
    }
  for (int s = lanes >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!live) return;
  const float inv = scale / sqrtf(ss / (float)valid + eps);
  for (int c = sub * W; c < V; c += lanes * W) {
    float f[W], g[W], k[W];
    load_f32<W>(src + c, f);
    load_f32<W>(gate + (size_t)r * ldg + h * V + c, g);
    load_f32<W>(w + c, k);
#pragma unroll
    for (int i = 0; i < W; ++i) f[i] *= inv * k[i] * sigmoid_f32(g[i]);
    store_row<T>(y + (size_t)r * ldy + h * V + c, f);
  }
}

template <typename T>
static int prepare(DeltaPrepArgs<T>& p, const int* cu, int n, cudaStream_t st) {
  int lanes = 1;
  while (lanes < 32 && lanes * kVec<T> < p.K) lanes *= 2;
  if (p.K > 256) return -6;
  p.lanes = lanes;
  const int tasks = ((p.G * lanes + 31) & ~31) + ((p.H * p.V / kVec<T> + 31) & ~31) + ((p.H * p.K / 4 + 31) & ~31) + p.H;
  p.run = cu == nullptr ? 1 : conv_run(p.rows, tasks, num_sms());
  p.keep = cu == nullptr && p.conv.taps > 1;
  dim3 grid((p.rows + p.run - 1) / p.run, (tasks + 127) / 128);
  if (p.conv.taps == 4) delta_prepare_kernel<T, 4><<<grid, 128, 0, st>>>(p);
  else delta_prepare_kernel<T, 0><<<grid, 128, 0, st>>>(p);
  return check_launch("delta_prepare_kernel");
}

template <typename T>
static int rule(const DeltaArgs<T>& a, int sequences, int longest, cudaStream_t st) {
  if (a.K <= 32) return launch_delta<T, 1>(a, sequences, longest, st);
  if (a.K <= 64) return launch_delta<T, 2>(a, sequences, longest, st);
  if (a.K <= 96) return launch_delta<T, 3>(a, sequences, longest, st);
  if (a.K <= 128) return launch_delta<T, 4>(a, sequences, longest, st);
  if (a.K <= 192) return launch_delta<T, 6>(a, sequences, longest, st);
  if (a.K <= 256) return launch_delta<T, 8>(a, sequences, longest, st);
  return -6;
}

}  // namespace icb

using namespace icb;

// x: columns [q: G x K | k: G x K | v: H x V] of rows with pitch ldx, K and V multiples of 8 (heads may be padded with
// zero columns); conv_w [taps][2 G K + H V] fp32 and conv_state [slots, taps - 1, 2 G K + H V] as in icb_short_conv,
// except that with cu != null the carried inputs are not updated here. beta_in: H logits, pitch ldbeta. a [rows, H x K]
// fp32 becomes exp(-exp(a_log) softplus(a + dt_bias)). q, k: fp32 unit vectors [rows, G x K], q times q_scale; qk
// [rows, G]; v [rows, H x V] and beta fp32 [rows, H]. K <= 256.
ICB_API int icb_delta_prepare(const void* x, long long ldx, const float* conv_w, void* conv_state, int taps,
                              const int* seqs, const int* pos, const int* cu, const void* beta_in, long long ldbeta,
                              float* a, const float* a_log, const float* dt_bias, float* q, float* k, float* qk, void* v,
                              float* beta, int rows, int G, int H, int K, int V, float q_scale, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (G < 1 || H % G || K % 8 || V % 8 || ldx % 8 || taps < 1) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  const int C = 2 * G * K + H * V;
  if (dtype == kBF16) {
    using T = __nv_bfloat16;
    DeltaPrepArgs<T> p{{(const T*)x, ldx, conv_w, nullptr, (T*)conv_state, seqs, pos, C, taps}, (const T*)beta_in, ldbeta, a,
                       a_log, dt_bias, q, k, qk, (T*)v, beta, rows, G, H, K, V, q_scale, 0, 0, 0};
    return prepare<T>(p, cu, 0, st);
  }
  if (dtype == kF32) {
    DeltaPrepArgs<float> p{{(const float*)x, ldx, conv_w, nullptr, (float*)conv_state, seqs, pos, C, taps},
                           (const float*)beta_in, ldbeta, a, a_log, dt_bias, q, k, qk, (float*)v, beta, rows, G, H, K, V,
                           q_scale, 0, 0, 0};
    return prepare<float>(p, cu, 0, st);
  }
  return -3;
}

// The recurrence over the rows of `sequences` sequences (cu [sequences + 1]; null: one row each). Operands as written by
// icb_delta_prepare; state [slots, H, V, K rounded up to a multiple of 32 (above 128: 64)] fp32; o [rows, H x V] fp32.
// `longest` bounds the rows of a sequence. dtype: v's.
ICB_API int icb_delta_rule(const float* q, const float* k, const float* g, const float* qk, const void* v,
                           const float* beta, float* state, float* o, const int* seqs, const int* pos, const int* cu,
                           int sequences, int longest, int G, int H, int K, int V, int dtype, void* stream) {
  if (sequences <= 0) return 0;
  if (G < 1 || H % G || H > 65535 || K % 8 || V % 8 || longest < 1 || (cu == nullptr && longest != 1)) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16) {
    DeltaArgs<__nv_bfloat16> a{q, k, g, qk, (const __nv_bfloat16*)v, beta, state, o, seqs, pos, cu, G, H, K, V};
    return rule<__nv_bfloat16>(a, sequences, longest, st);
  }
  if (dtype == kF32) {
    DeltaArgs<float> a{q, k, g, qk, (const float*)v, beta, state, o, seqs, pos, cu, G, H, K, V};
    return rule<float>(a, sequences, longest, st);
  }
  return -3;
}

// y [rows, pitch ldy] (dtype) = o / sqrt(mean(o^2 over a head's `valid` values) + eps) * w * sigmoid(gate) * scale for H
// heads of V values (a multiple of 8, zeros behind `valid`); o fp32 [rows, H x V], gate fp32 logits of pitch ldg, w [V].
ICB_API int icb_delta_output(const float* o, const float* gate, long long ldg, const float* w, float eps, float scale,
                             void* y, long long ldy, int rows, int H, int V, int valid, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (V % 8 || ldg % 4 || ldy % 8 || valid < 1 || valid > V) return -2;
  const int vec = dtype == kBF16 ? 8 : 4;
  int lanes = 1;
  while (lanes < 32 && lanes * vec < V) lanes *= 2;
  const long long threads = (long long)rows * H * lanes;
  const int blocks = (int)((threads + 255) / 256);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16)
    delta_output_kernel<__nv_bfloat16><<<blocks, 256, 0, st>>>(o, gate, ldg, w, eps, scale, (__nv_bfloat16*)y, ldy, rows, H, V,
                                                              valid, lanes);
  else if (dtype == kF32)
    delta_output_kernel<float><<<blocks, 256, 0, st>>>(o, gate, ldg, w, eps, scale, (float*)y, ldy, rows, H, V, valid, lanes);
  else return -3;
  return check_launch("delta_output_kernel");
}
