// Gated delta rule with a decay per key channel, fp32 state [dim x vdim] per head carried from batch to batch:
//
//   S <- g S          u = beta (v - S^T k)          S <- S + k u^T          o = S^T q
//
// Three kernels, each for any mixture of sequences (rows.cuh):
//   delta_prepare   short convolution + silu of q, k and v, unit norms of q and k, q . k, decay factors, beta
//   delta_rule      the recurrence
//   delta_output    RMS norm of a head's output, gain, output gate
//
// delta_rule: the columns of S do not depend on one another; a CTA takes some of them through a sequence with S in
// registers, while k, q, g and v rows of the next tile of tokens arrive by asynchronous copies.
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
constexpr int kPrepAhead = 2;         // rows whose loads are in flight per thread

// ROLES: 1 the q / k heads, 2 everything else, 3 both. Long batches run the two apart: the heads need many registers.
template <typename T, int TAPS, int ROLES>
__global__ void __launch_bounds__(128, ROLES == 2 ? 5 : 3) delta_prepare_kernel(const DeltaPrepArgs<T> p) {
  constexpr int W = kVec<T>;
  constexpr int S = sizeof(T) == 4 ? 2 : 1;           // pieces of a q / k head that one lane holds
  const ConvArgs<T>& a = p.conv;
  const int r0 = blockIdx.x * p.run, r1 = min(p.rows, r0 + p.run);
  if (r0 >= p.rows) return;
  // thread roles, each rounded up to whole warps: q / k heads, v channels, decay channels, beta
  int task = blockIdx.y * blockDim.x + threadIdx.x;
  const int n_qk = ROLES == 2 ? 0 : (p.G * p.lanes + 31) & ~31;
  const int n_v = (p.H * p.V / W + 31) & ~31, n_g = (p.H * p.K / 4 + 31) & ~31;
  const int most = (TAPS > 0 ? TAPS : a.taps) - 1;
  if (ROLES == 1 && task >= n_qk) return;
  if (task < n_qk + n_v) {
    const bool is_v = ROLES == 2 || (ROLES == 3 && task >= n_qk);
    if (is_v) task -= n_qk;
    const int head = is_v ? 0 : task / p.lanes, sub = is_v ? 0 : task - head * p.lanes;
    bool live[S];
    int ch[S];
    ConvLane<T, TAPS> lq[S], lk[S];
    int before = rows_before(a.seqs, r0, most), slot = a.seqs[r0];
#pragma unroll
    for (int e = 0; e < S; ++e) {
      const int c = (sub + e * p.lanes) * W;
      live[e] = is_v ? e == 0 && task < p.H * p.V / W : head < p.G && c < p.K;
      ch[e] = is_v ? 2 * p.G * p.K + task * W : head * p.K + c;
      if (live[e]) {
        lq[e].init(a, ch[e]);
        lq[e].refill(a, r0, before, slot, a.pos[r0]);
        if (!is_v) {
          lk[e].init(a, p.G * p.K + ch[e]);
          lk[e].refill(a, r0, before, slot, a.pos[r0]);
        }
      }
    }
    for (int g = r0; g < r1; g += kPrepAhead) {
      uint4 xq[kPrepAhead][S], xk[kPrepAhead][S];
#pragma unroll
      for (int i = 0; i < kPrepAhead; ++i)
#pragma unroll
        for (int e = 0; e < S; ++e)
          if (live[e] && g + i < r1) {
            xq[i][e] = lq[e].fetch(a, g + i);
            if (!is_v) xk[i][e] = lk[e].fetch(a, g + i);
          }
#pragma unroll
      for (int i = 0; i < kPrepAhead; ++i) {
        const int r = g + i;
        if (r >= r1) break;                      // the same for the whole block
        const int pos = a.pos[r];
        if (r > r0) {
          const int s = a.seqs[r];
          before = s == slot ? min(before + 1, most) : 0;
          if (s != slot) {
            slot = s;
#pragma unroll
            for (int e = 0; e < S; ++e)
              if (live[e]) {
                lq[e].refill(a, r, 0, slot, pos);
                if (!is_v) lk[e].refill(a, r, 0, slot, pos);
              }
          }
        }
        float x[S][W], y[S][W];
        if (is_v) {
          if (live[0]) {
            lq[0].row(a, xq[i][0], r, before, slot, pos, x[0]);
            store_row<T>(p.v + (size_t)r * p.H * p.V + task * W, x[0]);
            if (p.keep) conv_keep<T>(a, r, before, slot, pos, ch[0]);
          }
          continue;
        }
        float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int e = 0; e < S; ++e) {
          if (!live[e]) continue;
          lq[e].row(a, xq[i][e], r, before, slot, pos, x[e]);
          lk[e].row(a, xk[i][e], r, before, slot, pos, y[e]);
#pragma unroll
          for (int v = 0; v < W; ++v) {
            qq = fmaf(x[e][v], x[e][v], qq);
            kk = fmaf(y[e][v], y[e][v], kk);
            qk = fmaf(x[e][v], y[e][v], qk);
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
          for (int v = 0; v < W; ++v) { x[e][v] *= fq; y[e][v] *= fk; }
          store_f32<W>(p.q + (size_t)r * p.G * p.K + ch[e], x[e]);
          store_f32<W>(p.k + (size_t)r * p.G * p.K + ch[e], y[e]);
          if (e == 0 && sub == 0) p.qk[(size_t)r * p.G + head] = qk * fq * fk;
          if (p.keep) {
            conv_keep<T>(a, r, before, slot, pos, ch[e]);
            conv_keep<T>(a, r, before, slot, pos, p.G * p.K + ch[e]);
          }
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
        const float x = rate * softplus_of<T>(f[i] + bias[i]);
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

// One token for each of many sequences: bound by the bytes of the states. The key channels of a column lie on LN lanes:
// lane kl holds channels (j * LN + kl) * 4 .. + 3 for j < NJ, of four columns.
template <typename T, int LN, int NJ>
__global__ void __launch_bounds__(128) delta_one_kernel(const DeltaArgs<T> a) {
  constexpr int KP = LN * NJ * 4, VC = 4;
  const int r = blockIdx.x, h = blockIdx.y, kvh = h / (a.H / a.G);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % LN;
  const int col = (blockIdx.z * (blockDim.x >> 5) + warp) * (32 / LN * VC) + (lane / LN) * VC;
  const bool live = col < a.V;                                   // V is a multiple of 8: all four or none
  const bool fresh = a.pos[r] == 0;
  float* st = a.state + (((size_t)a.seqs[r] * a.H + h) * a.V + col) * KP + kl * 4;
  float s[VC][NJ][4];
#pragma unroll
  for (int c = 0; c < VC; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !fresh) u = *reinterpret_cast<const float4*>(st + (size_t)c * KP + j * LN * 4);
      s[c][j][0] = u.x; s[c][j][1] = u.y; s[c][j][2] = u.z; s[c][j][3] = u.w;
    }
  float k[NJ][4], sum[2 * VC];              // S^T k of the four columns, then S^T q, after the decay
#pragma unroll
  for (int i = 0; i < 2 * VC; ++i) sum[i] = 0.f;
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int ch = (j * LN + kl) * 4;
    float q[4], g[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) k[j][i] = q[i] = g[i] = 0.f;
    if (ch < a.K) {
      load_f32<4>(a.k + ((size_t)r * a.G + kvh) * a.K + ch, k[j]);
      load_f32<4>(a.q + ((size_t)r * a.G + kvh) * a.K + ch, q);
      load_f32<4>(a.g + ((size_t)r * a.H + h) * a.K + ch, g);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int c = 0; c < VC; ++c) {
        s[c][j][i] *= g[i];
        sum[c] = fmaf(s[c][j][i], k[j][i], sum[c]);
        sum[VC + c] = fmaf(s[c][j][i], q[i], sum[VC + c]);
      }
  }
  const float beta = a.beta[(size_t)r * a.H + h], qk = a.qk[(size_t)r * a.G + kvh];
#pragma unroll
  for (int i = 0; i < 2 * VC; ++i)
#pragma unroll
    for (int o = 1; o < LN; o <<= 1) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], o);
  if (!live) return;
#pragma unroll
  for (int c = 0; c < VC; ++c) {
    const float v = static_cast<float>(a.v[((size_t)r * a.H + h) * a.V + col + c]);
    const float u = beta * (v - sum[c]);
    if (kl == c) a.o[((size_t)r * a.H + h) * a.V + col + c] = fmaf(u, qk, sum[VC + c]);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
#pragma unroll
      for (int i = 0; i < 4; ++i) s[c][j][i] = fmaf(k[j][i], u, s[c][j][i]);
      *reinterpret_cast<float4*>(st + (size_t)c * KP + j * LN * 4) = make_float4(s[c][j][0], s[c][j][1], s[c][j][2], s[c][j][3]);
    }
  }
}

// Runs of tokens, four at a time. With G_i = g_1 .. g_i (products of decay factors, never a quotient), from the state S
// before the four tokens:
//   d_i = S^T (G_i k_i)        e_i = S^T (G_i q_i)                                     all eight in one pass over S
//   u_i = beta_i (v_i - d_i - sum_{j<i} A_ij u_j),      A_ij = (g_{j+1} .. g_i k_j) . k_i
//   o_i = e_i + sum_{j<=i} B_ij u_j,                    B_ij = (g_{j+1} .. g_i k_j) . q_i
//   S <- G_4 S + sum_j (g_{j+1} .. g_4 k_j) u_j^T
// A CTA takes some columns of a head through a sequence. Per tile of tokens it first turns k, q and g in shared memory into
// G_i k_i, G_i q_i and g_{j+1} .. g_4 k_j, one (group of four, channel) per thread, and sums A and B up. In the main pass
// the channels of a column are spread over 16 lanes (lane kl: channels (j * 16 + kl) * 4 .. + 3), a thread has four columns
// (what it loads of k, q and g from shared memory serves all of them: shared memory is the bound), and two channels make an
// fp32 pair. 32 sums (four tokens, d and e, four columns) meet in a transposing reduction that leaves two to every lane.
constexpr int kDeltaGroup = 4;
constexpr int kDeltaLanes = 16;
constexpr int kDeltaCols = 32 / kDeltaLanes * 4;       // columns of a warp

// Shared memory of one tile buffer in floats: k, q, g [tile][KP], beta and qk [tile], v [tile][cols] (T, 16-byte rows).
template <typename T>
__host__ __device__ inline int delta_vpitch(int cols) { return (cols * (int)sizeof(T) + 15) / 16 * 16 / (int)sizeof(T); }
template <typename T>
__host__ __device__ inline int delta_buf_floats(int kp, int cols, int tile) {
  return tile * (3 * kp + delta_vpitch<T>(cols) * (int)sizeof(T) / 4 + 2);
}

template <typename T, int NJ>         // 64 NJ >= K
__global__ void __launch_bounds__(256) delta_rule_kernel(const DeltaArgs<T> a, int tile, int state_pitch) {
  extern __shared__ __align__(16) float smem_f[];
  constexpr int LN = kDeltaLanes, KP = LN * NJ * 4, PK = KP / 4, PARTS = KP / 32;
  const SeqRows seq = seq_rows(a.cu, a.seqs, a.pos, blockIdx.x);
  if (seq.begin >= seq.end) return;
  const int h = blockIdx.y, kvh = h / (a.H / a.G);
  const int warps = blockDim.x >> 5, cols = warps * kDeltaCols;  // columns of this CTA
  const int col_base = blockIdx.z * cols, ncol = min(cols, a.V - col_base);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, kl = lane % LN;
  const int lc = warp * kDeltaCols + (lane / LN) * 4;            // first of this thread's four columns inside the CTA
  const int col = col_base + lc;
  const bool live = lc < ncol;                                   // V is a multiple of 8: all or none
  const int vpitch = delta_vpitch<T>(cols), buf_floats = delta_buf_floats<T>(KP, cols, tile);
  const int groups = tile / kDeltaGroup;
  auto vec = [&](int buf, int which) { return smem_f + buf * buf_floats + which * tile * KP; };
  auto sbuf = [&](int buf) { return smem_f + buf * buf_floats + 3 * tile * KP; };            // beta, then qk
  auto vbuf = [&](int buf) { return reinterpret_cast<T*>(smem_f + buf * buf_floats + tile * (3 * KP + 2)); };
  float* s_all = smem_f + 2 * buf_floats;                        // [groups][KP] G_4
  float* s_part = s_all + groups * KP;                           // [groups][PARTS][16] partial A, B
  float* s_mat = s_part + groups * PARTS * 16;                   // [groups][4][8]: row i of A, row i of B (zeros above)

  auto fetch = [&](int t0, int buf) {
    const int nt = min(tile, seq.end - t0);
    for (int i = threadIdx.x; i < nt * PK; i += blockDim.x) {
      const int t = i / PK, c = (i - t * PK) * 4;
      const size_t row = (size_t)(t0 + t);
      if (c < a.K) {
        cp_async16(vec(buf, 0) + t * KP + c, a.k + (row * a.G + kvh) * a.K + c);
        cp_async16(vec(buf, 1) + t * KP + c, a.q + (row * a.G + kvh) * a.K + c);
        cp_async16(vec(buf, 2) + t * KP + c, a.g + (row * a.H + h) * a.K + c);
      }
    }
    const int pv = ncol / kVec<T>;
    for (int i = threadIdx.x; i < nt * pv; i += blockDim.x) {
      const int t = i / pv, c = (i - t * pv) * kVec<T>;
      cp_async16(vbuf(buf) + t * vpitch + c, a.v + ((size_t)(t0 + t) * a.H + h) * a.V + col_base + c);
    }
    cp_async_commit();
    for (int t = threadIdx.x; t < nt; t += blockDim.x) {
      sbuf(buf)[t] = a.beta[(size_t)(t0 + t) * a.H + h];
      sbuf(buf)[tile + t] = a.qk[(size_t)(t0 + t) * a.G + kvh];
    }
    // tokens that change nothing fill the last group up
    const int fill = (kDeltaGroup - nt % kDeltaGroup) % kDeltaGroup;
    for (int i = threadIdx.x; i < fill * KP; i += blockDim.x) {
      const int at = nt * KP + i;
      vec(buf, 0)[at] = 0.f;
      vec(buf, 1)[at] = 0.f;
      vec(buf, 2)[at] = 1.f;
    }
    for (int i = threadIdx.x; i < fill * vpitch; i += blockDim.x) vbuf(buf)[nt * vpitch + i] = static_cast<T>(0.f);
    if (threadIdx.x < fill) sbuf(buf)[nt + threadIdx.x] = sbuf(buf)[tile + nt + threadIdx.x] = 0.f;
  };

  if (KP > a.K) {        // pad channels hold zeros in both buffers: the copies do not touch them
    const int pad = KP - a.K;
    for (int i = threadIdx.x; i < 2 * 3 * tile * pad; i += blockDim.x) {
      const int b = i / (3 * tile * pad), rest = i - b * (3 * tile * pad);
      vec(b, 0)[(rest / pad) * KP + a.K + rest % pad] = 0.f;
    }
    __syncthreads();
  }
  fetch(seq.begin, 0);

  Pair s[4][NJ][2];
  float* st = a.state + (((size_t)seq.slot * a.H + h) * a.V + col) * state_pitch + kl * 4;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
      if (live && !seq.fresh && j * LN * 4 + kl * 4 < state_pitch)
        u = *reinterpret_cast<const float4*>(st + (size_t)c * state_pitch + j * LN * 4);
      s[c][j][0] = pair_of(u.x, u.y);
      s[c][j][1] = pair_of(u.z, u.w);
    }
  // the sums that the reduction leaves to a lane: bits 0 and 1 the token, bit 2 e against d, bit 3 the pair of columns
  const int tok = (kl & 1) * 2 + ((kl >> 1) & 1), my = kl >> 3;
  const bool is_e = kl & 4;

  int buf = 0;
  for (int t0 = seq.begin; t0 < seq.end; t0 += tile, buf ^= 1) {
    const int nt = min(tile, seq.end - t0), ng = (nt + kDeltaGroup - 1) / kDeltaGroup;
    const bool more = t0 + tile < seq.end;
    if (more) {
      fetch(t0 + tile, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    for (int i = threadIdx.x; i < ng * KP; i += blockDim.x) {      // KP and the CTA are whole warps
      const int gr = i / KP, ch = i - gr * KP;
      float* pk = vec(buf, 0) + gr * kDeltaGroup * KP + ch;
      float* pq = vec(buf, 1) + gr * kDeltaGroup * KP + ch;
      float* pg = vec(buf, 2) + gr * kDeltaGroup * KP + ch;
      float k[4], q[4], g[4], sum[16];
#pragma unroll
      for (int m = 0; m < 4; ++m) { k[m] = pk[m * KP]; q[m] = pq[m * KP]; g[m] = pg[m * KP]; }
#pragma unroll
      for (int e = 0; e < 16; ++e) sum[e] = 0.f;
      float all = 1.f;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        all *= g[m];
        pk[m * KP] = all * k[m];
        pq[m * KP] = all * q[m];
        float w = k[m];
#pragma unroll
        for (int n = m + 1; n < 4; ++n) {
          w *= g[n];
          sum[n * (n - 1) / 2 + m] = w * k[n];
          sum[8 + n * (n - 1) / 2 + m] = w * q[n];
        }
        pg[m * KP] = w;
      }
      s_all[gr * KP + ch] = all;
      int off = 1;
#pragma unroll
      for (int half = 8; half > 0; half >>= 1, off <<= 1) {
        const bool up = lane & off;
#pragma unroll
        for (int e = 0; e < half; ++e) {
          const float keep = up ? sum[half + e] : sum[e], give = up ? sum[e] : sum[half + e];
          sum[e] = keep + __shfl_xor_sync(0xffffffffu, give, off);
        }
      }
      sum[0] += __shfl_xor_sync(0xffffffffu, sum[0], 16);
      // lane bits 0 .. 3 chose the bits 3 .. 0 of the index
      const int which = (lane & 1) * 8 + (lane & 2) * 2 + ((lane >> 1) & 2) + ((lane >> 3) & 1);
      if (lane < 16) s_part[(gr * PARTS + ch / 32) * 16 + which] = sum[0];
    }
    __syncthreads();
    for (int i = threadIdx.x; i < ng * 32; i += blockDim.x) {
      const int gr = i / 32, row = i / 8 % 4, at = i % 8, c = at % 4;
      float v = 0.f;
      if (c < row) {
#pragma unroll
        for (int p = 0; p < PARTS; ++p) v += s_part[(gr * PARTS + p) * 16 + (at / 4) * 8 + row * (row - 1) / 2 + c];
      } else if (c == row && at >= 4) {
        v = sbuf(buf)[tile + gr * 4 + row];
      }
      s_mat[i] = v;
    }
    __syncthreads();
    float* po = a.o + ((size_t)(t0 + tok) * a.H + h) * a.V + col + my * 2;
    for (int gr = 0; gr < ng; ++gr, po += (size_t)kDeltaGroup * a.H * a.V) {
      const float* pk = vec(buf, 0) + gr * kDeltaGroup * KP + kl * 4;
      const float* pq = vec(buf, 1) + gr * kDeltaGroup * KP + kl * 4;
      const float* pw = vec(buf, 2) + gr * kDeltaGroup * KP + kl * 4;
      float sum[32];                        // [token][d, e][column]
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        Pair d[4], e[4];
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const float4 k4 = *reinterpret_cast<const float4*>(pk + m * KP + j * LN * 4);
          const float4 q4 = *reinterpret_cast<const float4*>(pq + m * KP + j * LN * 4);
          const Pair kk[2] = {pair_of(k4.x, k4.y), pair_of(k4.z, k4.w)}, qq[2] = {pair_of(q4.x, q4.y), pair_of(q4.z, q4.w)};
#pragma unroll
          for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int c = 0; c < 4; ++c) {
              d[c] = j == 0 && i == 0 ? pair_mul(s[c][j][i], kk[i]) : pair_fma(s[c][j][i], kk[i], d[c]);
              e[c] = j == 0 && i == 0 ? pair_mul(s[c][j][i], qq[i]) : pair_fma(s[c][j][i], qq[i], e[c]);
            }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float2 x = pair_values(d[c]), y = pair_values(e[c]);
          sum[m * 8 + c] = x.x + x.y;
          sum[m * 8 + 4 + c] = y.x + y.y;
        }
      }
      int off = 1;
#pragma unroll
      for (int half = 16; half > 1; half >>= 1, off <<= 1) {
        const bool up = kl & off;
#pragma unroll
        for (int i = 0; i < half; ++i) {
          const float keep = up ? sum[half + i] : sum[i], give = up ? sum[i] : sum[half + i];
          sum[i] = keep + __shfl_xor_sync(0xffffffffu, give, off);
        }
      }
      const float4 ra = *reinterpret_cast<const float4*>(s_mat + (gr * 4 + tok) * 8);
      const float4 rb = *reinterpret_cast<const float4*>(s_mat + (gr * 4 + tok) * 8 + 4);
      const float rowa[4] = {ra.x, ra.y, ra.z, ra.w}, rowb[4] = {rb.x, rb.y, rb.z, rb.w};
      const float beta = sbuf(buf)[gr * 4 + tok];
      const T* pv = vbuf(buf) + (gr * 4 + tok) * vpitch + lc + my * 2;
      float want[2] = {-sum[0], -sum[1]}, o[2] = {sum[0], sum[1]}, u[4][4];
      if (live) {
        want[0] += static_cast<float>(pv[0]);
        want[1] += static_cast<float>(pv[1]);
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const int from = (m >> 1) | ((m & 1) << 1);       // the lanes where beta * want is u of token m
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          const float mine = beta * want[c];
          u[m][c] = __shfl_sync(0xffffffffu, mine, from, LN);
          u[m][2 + c] = __shfl_sync(0xffffffffu, mine, from + 8, LN);
          const float um = my ? u[m][2 + c] : u[m][c];
          want[c] = fmaf(-rowa[m], um, want[c]);
          o[c] = fmaf(rowb[m], um, o[c]);
        }
      }
      if (is_e && live && gr * 4 + tok < nt) *reinterpret_cast<float2*>(po) = make_float2(o[0], o[1]);
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const float4 g4 = *reinterpret_cast<const float4*>(s_all + gr * KP + kl * 4 + j * LN * 4);
        const Pair gg[2] = {pair_of(g4.x, g4.y), pair_of(g4.z, g4.w)};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          s[c][j][0] = pair_mul(s[c][j][0], gg[0]);
          s[c][j][1] = pair_mul(s[c][j][1], gg[1]);
        }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          const float4 w4 = *reinterpret_cast<const float4*>(pw + m * KP + j * LN * 4);
          const Pair ww[2] = {pair_of(w4.x, w4.y), pair_of(w4.z, w4.w)};
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const Pair uu = pair_of(u[m][c], u[m][c]);
            s[c][j][0] = pair_fma(ww[0], uu, s[c][j][0]);
            s[c][j][1] = pair_fma(ww[1], uu, s[c][j][1]);
          }
        }
      }
    }
    if (more) __syncthreads();            // this buffer is the next but one fetch's target, and the sums are rewritten
  }
  if (live) {
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        if (j * LN * 4 + kl * 4 >= state_pitch) continue;
        const float2 x = pair_values(s[c][j][0]), y = pair_values(s[c][j][1]);
        *reinterpret_cast<float4*>(st + (size_t)c * state_pitch + j * LN * 4) = make_float4(x.x, x.y, y.x, y.y);
      }
  }
}

template <typename T, int NJ>
static int launch_delta(const DeltaArgs<T>& a, int sequences, int longest, int state_pitch, cudaStream_t st) {
  // wide CTAs share the work on k, q and g among more columns; narrower ones if that leaves SMs without a CTA
  int warps = 8;
  while (warps > 1 && ((warps / 2) * kDeltaCols >= a.V ||
                       (long long)sequences * a.H * ((a.V + warps * kDeltaCols - 1) / (warps * kDeltaCols)) < num_sms() * 3 / 4))
    warps >>= 1;
  constexpr int KP = kDeltaLanes * NJ * 4;
  const int cols = warps * kDeltaCols;
  int tile = (longest + kDeltaGroup - 1) / kDeltaGroup * kDeltaGroup;
  const int most = warps >= 4 ? 16 : 8;
  if (tile > most) tile = most;
  const int groups = tile / kDeltaGroup;
  const size_t smem = 4 * (2 * (size_t)delta_buf_floats<T>(KP, cols, tile) + groups * (KP + KP / 32 * 16 + 32));
  auto kern = delta_rule_kernel<T, NJ>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return -(int)e;
  }
  dim3 grid(sequences, a.H, (a.V + cols - 1) / cols);
  kern<<<grid, warps * 32, smem, st>>>(a, tile, state_pitch);
  return check_launch("delta_rule_kernel");
}

template <typename T, int LN, int NJ>
static int launch_delta_one(const DeltaArgs<T>& a, int rows, cudaStream_t st) {
  constexpr int WC = 32 / LN * 4;
  int warps = 4;
  while (warps > 1 && warps / 2 * WC >= a.V) warps >>= 1;
  dim3 grid(rows, a.H, (a.V + warps * WC - 1) / (warps * WC));
  delta_one_kernel<T, LN, NJ><<<grid, warps * 32, 0, st>>>(a);
  return check_launch("delta_one_kernel");
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
static int prepare(DeltaPrepArgs<T>& p, const int* cu, cudaStream_t st) {
  int lanes = 1;
  while (lanes < 32 && lanes * kVec<T> < p.K) lanes *= 2;
  if (p.K > 256) return -6;
  p.lanes = lanes;
  const int heads = (p.G * lanes + 31) & ~31;
  const int others = ((p.H * p.V / kVec<T> + 31) & ~31) + ((p.H * p.K / 4 + 31) & ~31) + p.H;
  p.keep = cu == nullptr && p.conv.taps > 1;
  if (cu != nullptr && p.rows >= 256 && p.conv.taps == 4) {
    p.run = conv_run(p.rows, heads, num_sms(), 3 * 128);
    dim3 g1((p.rows + p.run - 1) / p.run, (heads + 127) / 128);
    delta_prepare_kernel<T, 4, 1><<<g1, 128, 0, st>>>(p);
    p.run = conv_run(p.rows, others, num_sms(), 5 * 128);
    dim3 g2((p.rows + p.run - 1) / p.run, (others + 127) / 128);
    delta_prepare_kernel<T, 4, 2><<<g2, 128, 0, st>>>(p);
    return check_launch("delta_prepare_kernel");
  }
  p.run = cu == nullptr ? 1 : conv_run(p.rows, heads + others, num_sms(), 3 * 128);
  dim3 grid((p.rows + p.run - 1) / p.run, (heads + others + 127) / 128);
  if (p.conv.taps == 4) delta_prepare_kernel<T, 4, 3><<<grid, 128, 0, st>>>(p);
  else delta_prepare_kernel<T, 0, 3><<<grid, 128, 0, st>>>(p);
  return check_launch("delta_prepare_kernel");
}

template <typename T>
static int rule(const DeltaArgs<T>& a, int sequences, int longest, cudaStream_t st) {
  const int pitch = a.K <= 128 ? (a.K + 31) / 32 * 32 : (a.K + 63) / 64 * 64;
  if (a.K > 256) return -6;
  if (a.cu == nullptr) {
    switch (pitch) {
      case 32: return launch_delta_one<T, 8, 1>(a, sequences, st);
      case 64: return launch_delta_one<T, 16, 1>(a, sequences, st);
      case 96: return launch_delta_one<T, 8, 3>(a, sequences, st);
      case 128: return launch_delta_one<T, 16, 2>(a, sequences, st);
      case 192: return launch_delta_one<T, 16, 3>(a, sequences, st);
      default: return launch_delta_one<T, 16, 4>(a, sequences, st);
    }
  }
  if (a.K <= 64) return launch_delta<T, 1>(a, sequences, longest, pitch, st);
  if (a.K <= 128) return launch_delta<T, 2>(a, sequences, longest, pitch, st);
  if (a.K <= 192) return launch_delta<T, 3>(a, sequences, longest, pitch, st);
  return launch_delta<T, 4>(a, sequences, longest, pitch, st);
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
    return prepare<T>(p, cu, st);
  }
  if (dtype == kF32) {
    DeltaPrepArgs<float> p{{(const float*)x, ldx, conv_w, nullptr, (float*)conv_state, seqs, pos, C, taps},
                           (const float*)beta_in, ldbeta, a, a_log, dt_bias, q, k, qk, (float*)v, beta, rows, G, H, K, V,
                           q_scale, 0, 0, 0};
    return prepare<float>(p, cu, st);
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
