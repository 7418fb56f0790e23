// Helpers for kernels that walk token rows: vector loads and stores of bf16 / fp32 rows as fp32, activations in full
// precision, asynchronous 16-byte copies, and the short causal convolution over a batch of sequences.
#pragma once

#include "ptx.cuh"

namespace icb {

// Elements of one 16-byte access.
template <typename T>
constexpr int kVec = 16 / (int)sizeof(T);

template <typename T>
__device__ __forceinline__ void load_row(const T* p, float (&f)[kVec<T>]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  if constexpr (sizeof(T) == 4) {
    f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
  } else {
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
  }
}
template <typename T>
__device__ __forceinline__ void store_row(T* p, const float (&f)[kVec<T>]) {
  if constexpr (sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  } else {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]),
                                              pack_bf16x2(f[6], f[7]));
  }
}
template <int V>
__device__ __forceinline__ void load_f32(const float* p, float (&f)[V]) {
#pragma unroll
  for (int i = 0; i < V; i += 4) {
    const float4 u = *reinterpret_cast<const float4*>(p + i);
    f[i] = u.x; f[i + 1] = u.y; f[i + 2] = u.z; f[i + 3] = u.w;
  }
}
template <int V>
__device__ __forceinline__ void store_f32(float* p, const float (&f)[V]) {
#pragma unroll
  for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(f[i], f[i + 1], f[i + 2], f[i + 3]);
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem)), "l"(gmem) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// ----------------------------------------------------------------------------
// Rows of several sequences: rows of a sequence are adjacent and in order, row r belongs to sequence slot seqs[r] at
// position pos[r]. With cu != null sequence i of the batch has rows [cu[i], cu[i + 1]); without it every row is a
// sequence of its own (one more token for each).
// ----------------------------------------------------------------------------
struct SeqRows {
  int begin, end, slot;
  bool fresh;                  // starts at its first token: whatever the slot holds is somebody else's
};
__device__ __forceinline__ SeqRows seq_rows(const int* cu, const int* seqs, const int* pos, int i) {
  SeqRows s;
  s.begin = cu != nullptr ? cu[i] : i;
  s.end = cu != nullptr ? cu[i + 1] : i + 1;
  s.slot = 0;
  s.fresh = true;
  if (s.begin < s.end) {
    s.slot = seqs[s.begin];
    s.fresh = pos[s.begin] == 0;
  }
  return s;
}

// ----------------------------------------------------------------------------
// Short causal convolution, per channel: out[t] = bias + sum_j w[taps - 1 - j] x[t - j], zeros before a sequence's
// first token. state[slot][taps - 1][C] holds the inputs before the batch's first row of a sequence, oldest first.
// ----------------------------------------------------------------------------
template <typename T>
struct ConvArgs {
  const T* x;                  // [rows, pitch ldx]
  long long ldx;
  const float* w;              // [taps][C], the last one belongs to the current token
  const float* bias;           // [C] or null
  T* state;                    // [slots, taps - 1, C]
  const int* seqs;
  const int* pos;
  int C, taps;
};

// Rows of the same sequence right before row r in this batch, counted up to taps - 1.
__device__ __forceinline__ int rows_before(const int* seqs, int r, int most) {
  int n = 0;
  while (n < most && r - n - 1 >= 0 && seqs[r - n - 1] == seqs[r]) ++n;
  return n;
}

// The input j tokens before row r (0 = the row itself); `before` = rows_before(r).
template <typename T>
__device__ __forceinline__ void conv_input(const ConvArgs<T>& a, int r, int before, int slot, int pos, int j, int ch,
                                           float (&f)[kVec<T>]) {
  if (j <= before) {
    load_row<T>(a.x + (size_t)(r - j) * a.ldx + ch, f);
  } else if (pos - j >= 0) {
    load_row<T>(a.state + ((size_t)slot * (a.taps - 1) + (a.taps - 1 - (j - before))) * a.C + ch, f);
  } else {
#pragma unroll
    for (int v = 0; v < kVec<T>; ++v) f[v] = 0.f;
  }
}

// Convolution and silu of kVec<T> channels of row r. TAPS > 0 fixes the number of taps and takes the weights of `w`
// from registers (load_conv_weights); 0 reads both at run time.
template <typename T, int TAPS>
struct ConvWeights {
  float w[TAPS > 0 ? TAPS : 1][kVec<T>];
};
template <typename T, int TAPS>
__device__ __forceinline__ void load_conv_weights(const ConvArgs<T>& a, int ch, ConvWeights<T, TAPS>& k) {
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_f32<kVec<T>>(a.w + (size_t)(TAPS - 1 - j) * a.C + ch, k.w[j]);
  }
}
template <typename T, int TAPS>
__device__ __forceinline__ void conv_silu_row(const ConvArgs<T>& a, const ConvWeights<T, TAPS>& k, int r, int before,
                                              int slot, int pos, int ch, float (&out)[kVec<T>]) {
  constexpr int V = kVec<T>;
  if (a.bias != nullptr) load_f32<V>(a.bias + ch, out);
  else {
#pragma unroll
    for (int v = 0; v < V; ++v) out[v] = 0.f;
  }
  const int taps = TAPS > 0 ? TAPS : a.taps;
#pragma unroll
  for (int j = 0; j < taps; ++j) {
    float x[V];
    conv_input<T>(a, r, before, slot, pos, j, ch, x);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int v = 0; v < V; ++v) out[v] = fmaf(k.w[j][v], x[v], out[v]);
    } else {
      float w[V];
      load_f32<V>(a.w + (size_t)(taps - 1 - j) * a.C + ch, w);
#pragma unroll
      for (int v = 0; v < V; ++v) out[v] = fmaf(w[v], x[v], out[v]);
    }
  }
#pragma unroll
  for (int v = 0; v < V; ++v) out[v] = silu_f32(out[v]);
}

// The inputs that a sequence's next token needs, from its last row r of this batch. Entry e takes what is newer than
// itself only, so one thread may do this in place in ascending order.
template <typename T>
__device__ __forceinline__ void conv_keep(const ConvArgs<T>& a, int r, int before, int slot, int pos, int ch) {
  for (int e = 0; e + 1 < a.taps; ++e) {
    float f[kVec<T>];
    conv_input<T>(a, r, before, slot, pos, a.taps - 2 - e, ch, f);
    store_row<T>(a.state + ((size_t)slot * (a.taps - 1) + e) * a.C + ch, f);
  }
}

// How many consecutive rows a thread takes: long runs keep the taps in L1, but the machine should be full first.
inline int conv_run(long long rows, long long threads_per_row, int sms) {
  const long long fill = (long long)sms * 2048;
  long long run = rows * threads_per_row / fill;
  if (run < 1) run = 1;
  if (run > 32) run = 32;
  return (int)run;
}

}  // namespace icb
