// Attention with grouped key / value heads over a paged cache, the parts around the tensor-core kernels:
//
//  * rope_cache  : one pass over the packed projection of a batch: rotates the heads of q and k in place (partial rotary,
//                  pairs (i, i + dims / 2)), writes the rotated keys and the values to their cache rows
//                  and turns the gate logits into factors.
//  * attend_rows : one query row of one head per CTA against its visible cache rows, any head sizes, bf16 or fp32, all
//                  arithmetic in fp32. It serves fp32 models and shapes that the tensor-core kernels do not take.
#include "host_common.h"
#include "rows.cuh"
#include "visible.cuh"

namespace icb {

template <typename T>
struct RopeCacheArgs {
  T* z;                     // [rows, ldz]: [q: H x KD | k: G x KD | v: G x VD | gate logits: H]
  long long ldz;
  T* k_cache;               // [slots, G x KD]
  T* v_cache;               // [slots, G x VD]
  const long long* slots;   // cache row of a token, negative: none
  const int* pos;
  const double* freq;       // [half] radians per position
  float* gate;              // [rows, H] or null
  float gate_scale;
  int H, G, KD, VD, half;   // half: rotated pairs per head
};

constexpr int kRopeThreads = 128;

template <typename T, int W>      // W: elements per access of the rotated part
__global__ void __launch_bounds__(kRopeThreads) rope_cache_kernel(const RopeCacheArgs<T> a) {
  extern __shared__ float cs[];   // [half] cos, [half] sin
  const int r = blockIdx.x;
  T* z = a.z + (size_t)r * a.ldz;
  const double p = (double)a.pos[r];
  for (int i = threadIdx.x; i < a.half; i += kRopeThreads) {
    // an fp32 product loses position * 2^-24 radians, which grows along a sequence: product and reduction to one turn in
    // fp64, once per row and pair
    double turn = p * a.freq[i] * 0.15915494309189535;
    turn -= rint(turn);
    float s, c;
    sincosf((float)(turn * 6.283185307179586), &s, &c);
    cs[i] = c;
    cs[a.half + i] = s;
  }
  __syncthreads();
  const long long slot = a.slots[r];
  T* kc = slot >= 0 ? a.k_cache + (size_t)slot * a.G * a.KD : nullptr;
  T* vc = slot >= 0 ? a.v_cache + (size_t)slot * a.G * a.VD : nullptr;
  const int pairs = a.half / W;
  for (int idx = threadIdx.x; idx < (a.H + a.G) * pairs; idx += kRopeThreads) {
    const int h = idx / pairs, i = (idx - h * pairs) * W;
    T* x = z + (size_t)h * a.KD + i;
    float u[W], v[W];
    if constexpr (W == kVec<T>) {
      load_row<T>(x, u);
      load_row<T>(x + a.half, v);
    } else {
      u[0] = static_cast<float>(x[0]);
      v[0] = static_cast<float>(x[a.half]);
    }
#pragma unroll
    for (int e = 0; e < W; ++e) {
      const float c = cs[i + e], s = cs[a.half + i + e], uu = u[e], vv = v[e];
      u[e] = uu * c - vv * s;
      v[e] = vv * c + uu * s;
    }
    T* out = h >= a.H && kc != nullptr ? kc + (size_t)(h - a.H) * a.KD + i : nullptr;
    if constexpr (W == kVec<T>) {
      store_row<T>(x, u);
      store_row<T>(x + a.half, v);
      if (out != nullptr) {
        store_row<T>(out, u);
        store_row<T>(out + a.half, v);
      }
    } else {
      const T ut = static_cast<T>(u[0]), vt = static_cast<T>(v[0]);
      x[0] = ut;
      x[a.half] = vt;
      if (out != nullptr) {
        out[0] = ut;
        out[a.half] = vt;
      }
    }
  }
  if (kc != nullptr) {
    const T* k = z + (size_t)a.H * a.KD;
    const int rest = a.KD - 2 * a.half;
    for (int idx = threadIdx.x; idx < a.G * rest; idx += kRopeThreads) {
      const int c = (idx / rest) * a.KD + 2 * a.half + idx % rest;
      kc[c] = k[c];
    }
    const T* v = k + (size_t)a.G * a.KD;
    constexpr int V = kVec<T>;
    for (int idx = threadIdx.x; idx < a.G * a.VD / V; idx += kRopeThreads)
      reinterpret_cast<uint4*>(vc)[idx] = reinterpret_cast<const uint4*>(v)[idx];
  }
  if (a.gate != nullptr) {
    const T* g = z + (size_t)(a.H + a.G) * a.KD + (size_t)a.G * a.VD;
    for (int h = threadIdx.x; h < a.H; h += kRopeThreads)
      a.gate[(size_t)r * a.H + h] = a.gate_scale * sigmoid_f32(static_cast<float>(g[h]));
  }
}

template <typename T>
static int launch_rope_cache(const RopeCacheArgs<T>& a, int rows, cudaStream_t st) {
  const size_t smem = 2 * (size_t)a.half * sizeof(float);
  if (a.half % kVec<T> == 0) rope_cache_kernel<T, kVec<T>><<<rows, kRopeThreads, smem, st>>>(a);
  else rope_cache_kernel<T, 1><<<rows, kRopeThreads, smem, st>>>(a);
  return check_launch("rope_cache_kernel");
}

// ---------------------------------------------------------------------------------------------------------
template <typename T>
struct AttendRowsArgs {
  const T* q;               // [rows, ldq], heads KD apart
  long long ldq;
  const T* k_cache;         // [slots, G x KD]
  const T* v_cache;         // [slots, G x VD]
  const int* table;         // [sequences, max_blocks]
  const int* seqs;
  const int* pos;
  const float* gate;        // [rows, H] or null
  T* out;                   // [rows, ldo], heads VD apart
  long long ldo;
  int H, G, KD, VD, block_size, max_blocks;
  Visible see;
  float scale;
};

constexpr int kAttendThreads = 128;
constexpr int kAttendMaxOut = 8;    // output columns per thread

template <typename T>
__global__ void __launch_bounds__(kAttendThreads) attend_rows_kernel(const AttendRowsArgs<T> a) {
  extern __shared__ __align__(16) float sq[];       // [KD]
  __shared__ float sp[kAttendThreads];
  __shared__ long long srow[kAttendThreads];
  __shared__ float red[2][4];
  constexpr int V = kVec<T>;
  const int r = blockIdx.x, h = blockIdx.y, g = h / (a.H / a.G);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const T* q = a.q + (size_t)r * a.ldq + (size_t)h * a.KD;
  for (int i = tid; i < a.KD; i += kAttendThreads) sq[i] = static_cast<float>(q[i]) * a.scale;
  const int pos = a.pos[r], first = first_visible(a.see, pos);
  const int* pages = a.table + (size_t)a.seqs[r] * a.max_blocks;
  float m = -INFINITY, l = 0.f, acc[kAttendMaxOut];
#pragma unroll
  for (int i = 0; i < kAttendMaxOut; ++i) acc[i] = 0.f;
  __syncthreads();
  for (int t0 = first; t0 <= pos; t0 += kAttendThreads) {
    const int t = t0 + tid, n = min(kAttendThreads, pos + 1 - t0);
    float s = -INFINITY;
    if (t <= pos) {
      const long long row = (long long)pages[t / a.block_size] * a.block_size + t % a.block_size;
      srow[tid] = row;
      const T* k = a.k_cache + (size_t)row * a.G * a.KD + (size_t)g * a.KD;
      float s0 = 0.f, s1 = 0.f;
      for (int c = 0; c < a.KD; c += V) {
        float f[V];
        load_row<T>(k + c, f);
#pragma unroll
        for (int e = 0; e < V; e += 2) {
          s0 = fmaf(f[e], sq[c + e], s0);
          s1 = fmaf(f[e + 1], sq[c + e + 1], s1);
        }
      }
      s = s0 + s1;
    }
    const float wm = warp_max(s);
    if (lane == 0) red[0][warp] = wm;
    __syncthreads();
    const float m_new = fmaxf(m, fmaxf(fmaxf(red[0][0], red[0][1]), fmaxf(red[0][2], red[0][3])));
    const float p = expf(s - m_new), corr = expf(m - m_new);
    sp[tid] = p;
    const float ws = warp_sum(p);
    if (lane == 0) red[1][warp] = ws;
    __syncthreads();
    l = l * corr + red[1][0] + red[1][1] + red[1][2] + red[1][3];
    m = m_new;
#pragma unroll
    for (int i = 0; i < kAttendMaxOut; ++i) {
      const int d = i * kAttendThreads + tid;
      if (d >= a.VD) break;
      float o = acc[i] * corr;
      const T* v = a.v_cache + (size_t)g * a.VD + d;
      for (int j = 0; j < n; ++j) o = fmaf(sp[j], static_cast<float>(v[(size_t)srow[j] * a.G * a.VD]), o);
      acc[i] = o;
    }
    __syncthreads();
  }
  const float inv = (a.gate != nullptr ? a.gate[(size_t)r * a.H + h] : 1.f) / l;
#pragma unroll
  for (int i = 0; i < kAttendMaxOut; ++i) {
    const int d = i * kAttendThreads + tid;
    if (d < a.VD) a.out[(size_t)r * a.ldo + (size_t)h * a.VD + d] = static_cast<T>(acc[i] * inv);
  }
}

}  // namespace icb

using namespace icb;

// z [rows, ldz] (bf16 or fp32): [q: H x KD | k: G x KD | v: G x VD | H gate logits]. The first 2 * half elements of every
// q and k head rotate in place by pos * freq (fp64 [half]; pairs i, i + half); keys and values go to rows `slots` (int64, negative:
// skip) of the caches; gate (fp32 [rows, H], optional) = gate_scale * sigmoid(logit). KD, VD, ldz: multiples of 8.
ICB_API int icb_rope_cache(void* z, long long ldz, void* k_cache, void* v_cache, const long long* slots, const int* pos,
                           const double* freq, int half, float* gate, float gate_scale, int rows, int H, int G, int KD,
                           int VD, int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (G < 1 || H % G || KD % 8 || VD % 8 || ldz % 8 || half < 0 || 2 * half > KD || half > 4096) return -2;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16) {
    using T = __nv_bfloat16;
    RopeCacheArgs<T> a{(T*)z, ldz, (T*)k_cache, (T*)v_cache, slots, pos, freq, gate, gate_scale, H, G, KD, VD, half};
    return launch_rope_cache<T>(a, rows, st);
  }
  if (dtype == kF32) {
    RopeCacheArgs<float> a{(float*)z, ldz, (float*)k_cache, (float*)v_cache, slots, pos, freq, gate, gate_scale, H, G, KD, VD, half};
    return launch_rope_cache<float>(a, rows, st);
  }
  return -3;
}

// out [rows, ldo], heads VD apart: softmax attention of query rows (q [rows, ldq], heads KD apart) over the cache rows of
// sequence seqs[r] up to position pos[r] that `window` (tokens, 0: none) and `chunk` (0: none) leave visible, times the
// factor gate[r, h] if given. KD a multiple of 8, VD <= 1024.
ICB_API int icb_attend_rows(const void* q, long long ldq, const void* k_cache, const void* v_cache, const int* table,
                            int max_blocks, int block_size, const int* seqs, const int* pos, const float* gate, void* out,
                            long long ldo, int rows, int H, int G, int KD, int VD, int window, int chunk, float scale,
                            int dtype, void* stream) {
  if (rows <= 0) return 0;
  if (G < 1 || H % G || H > 65535 || KD % 8 || VD < 1 || block_size < 1) return -2;
  if (VD > kAttendThreads * kAttendMaxOut || KD > 8192) return -6;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  dim3 grid(rows, H);
  const size_t smem = (size_t)KD * sizeof(float);
  const Visible see{window > 0 ? window : 0, chunk > 0 ? chunk : 0};
  if (dtype == kBF16) {
    using T = __nv_bfloat16;
    AttendRowsArgs<T> a{(const T*)q, ldq, (const T*)k_cache, (const T*)v_cache, table, seqs, pos, gate, (T*)out, ldo, H, G,
                        KD, VD, block_size, max_blocks, see, scale};
    attend_rows_kernel<T><<<grid, kAttendThreads, smem, st>>>(a);
  } else if (dtype == kF32) {
    AttendRowsArgs<float> a{(const float*)q, ldq, (const float*)k_cache, (const float*)v_cache, table, seqs, pos, gate,
                            (float*)out, ldo, H, G, KD, VD, block_size, max_blocks, see, scale};
    attend_rows_kernel<float><<<grid, kAttendThreads, smem, st>>>(a);
  } else {
    return -3;
  }
  return check_launch("attend_rows_kernel");
}
