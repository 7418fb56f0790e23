// Helpers for kernels that walk token rows: vector loads and stores of bf16 / fp32 rows as fp32, activations in full
// precision, asynchronous 16-byte copies, and the short causal convolution over a batch of sequences.
#pragma once

#include "ptx.cuh"

namespace icb {

// Elements of one 16-byte access.
template <typename T>
constexpr int kVec = 16 / (int)sizeof(T);

template <typename T>
__device__ __forceinline__ void unpack_row(const uint4 u, float (&f)[kVec<T>]) {
  if constexpr (sizeof(T) == 4) {
    f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
  } else {
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
  }
}
template <typename T>
__device__ __forceinline__ void load_row(const T* p, float (&f)[kVec<T>]) {
  unpack_row<T>(*reinterpret_cast<const uint4*>(p), f);
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
// An activation of a 16-bit tensor: fast exp and division. Of an fp32 tensor: full precision.
template <typename T>
__device__ __forceinline__ float silu_of(float x) {
  if constexpr (sizeof(T) == 4) return silu_f32(x);
  return __fdividef(x, 1.f + __expf(-x));
}
// log(1 + exp(x)). The 16-bit models' form sums log(1 + e) = 2 artanh(e / (2 + e)) for e = exp(-|x|) <= 1 as a series
// (argument at most 1/3, first term left out below 1.5e-7 of the sum).
template <typename T>
__device__ __forceinline__ float softplus_of(float x) {
  if constexpr (sizeof(T) == 4) return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
  const float e = __expf(-fabsf(x)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = fmaf(q, 1.f / 11.f, 1.f / 9.f);
  p = fmaf(q, p, 1.f / 7.f);
  p = fmaf(q, p, 1.f / 5.f);
  p = fmaf(q, p, 1.f / 3.f);
  p = fmaf(q, p, 1.f);
  return fmaxf(x, 0.f) + 2.f * s * p;
}

// Two fp32 values in a register pair: one instruction multiplies and adds both.
struct Pair {
  unsigned long long v;
};
__device__ __forceinline__ Pair pair_of(float lo, float hi) {
  Pair p;
  asm("mov.b64 %0, {%1, %2};" : "=l"(p.v) : "f"(lo), "f"(hi));
  return p;
}
__device__ __forceinline__ float2 pair_values(Pair p) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(p.v));
  return f;
}
__device__ __forceinline__ Pair pair_mul(Pair a, Pair b) {
  Pair d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d.v) : "l"(a.v), "l"(b.v));
  return d;
}
__device__ __forceinline__ Pair pair_fma(Pair a, Pair b, Pair c) {
  Pair d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return d;
}

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

// The same values as they are stored: one 16-byte piece.
template <typename T>
__device__ __forceinline__ uint4 conv_piece(const ConvArgs<T>& a, int r, int before, int slot, int pos, int j, int ch) {
  if (j <= before) return *reinterpret_cast<const uint4*>(a.x + (size_t)(r - j) * a.ldx + ch);
  if (pos - j >= 0)
    return *reinterpret_cast<const uint4*>(a.state + ((size_t)slot * (a.taps - 1) + (a.taps - 1 - (j - before))) * a.C + ch);
  return make_uint4(0u, 0u, 0u, 0u);
}

// Convolution and silu of kVec<T> neighbouring channels along consecutive rows. TAPS > 0: the weights and the last
// TAPS - 1 inputs stay in registers, a row costs one load. TAPS == 0: any number of taps, everything read per row.
template <typename T, int TAPS>
struct ConvLane {
  static constexpr int V = kVec<T>;
  static constexpr int H = TAPS > 1 ? TAPS - 1 : 1;
  float w[TAPS > 0 ? TAPS : 1][V];      // [j]: of the input j tokens back
  uint4 past[H];                        // [j]: the input j + 1 tokens back
  int ch;

  __device__ __forceinline__ void init(const ConvArgs<T>& a, int channel) {
    ch = channel;
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) load_f32<V>(a.w + (size_t)(TAPS - 1 - j) * a.C + ch, w[j]);
    }
  }
  // before row r, when the row before it was not the last one this lane has seen of the same sequence
  __device__ __forceinline__ void refill(const ConvArgs<T>& a, int r, int before, int slot, int pos) {
    if constexpr (TAPS > 1) {
#pragma unroll
      for (int j = 1; j < TAPS; ++j) past[j - 1] = conv_piece<T>(a, r, before, slot, pos, j, ch);
    }
  }
  __device__ __forceinline__ uint4 fetch(const ConvArgs<T>& a, int r) const {
    return *reinterpret_cast<const uint4*>(a.x + (size_t)r * a.ldx + ch);
  }
  __device__ __forceinline__ void row(const ConvArgs<T>& a, uint4 x, int r, int before, int slot, int pos, float (&out)[V]) {
    if (a.bias != nullptr) load_f32<V>(a.bias + ch, out);
    else {
#pragma unroll
      for (int v = 0; v < V; ++v) out[v] = 0.f;
    }
    float f[V];
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int j = TAPS - 1; j > 0; --j) {
        unpack_row<T>(past[j - 1], f);
#pragma unroll
        for (int v = 0; v < V; ++v) out[v] = fmaf(w[j][v], f[v], out[v]);
        if (j > 1) past[j - 1] = past[j - 2];
      }
      unpack_row<T>(x, f);
#pragma unroll
      for (int v = 0; v < V; ++v) out[v] = fmaf(w[0][v], f[v], out[v]);
      if constexpr (TAPS > 1) past[0] = x;
    } else {
      for (int j = 0; j < a.taps; ++j) {
        conv_input<T>(a, r, before, slot, pos, j, ch, f);
        load_f32<V>(a.w + (size_t)(a.taps - 1 - j) * a.C + ch, w[0]);
#pragma unroll
        for (int v = 0; v < V; ++v) out[v] = fmaf(w[0][v], f[v], out[v]);
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) out[v] = silu_of<T>(out[v]);
  }
};

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

// How many consecutive rows a thread takes: long runs share the weights and the first inputs, but the machine
// (`resident` threads per SM) should be full two times over first.
inline int conv_run(long long rows, long long threads_per_row, int sms, int resident) {
  long long run = rows * threads_per_row / (2LL * sms * resident);
  if (run < 1) run = 1;
  if (run > 64) run = 64;
  return (int)run;
}

}  // namespace icb
