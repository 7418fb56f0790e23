// Short causal convolution over time with silu, for rows of many sequences (see rows.cuh), and the update of the
// inputs that every sequence carries along.
#include "host_common.h"
#include "rows.cuh"

namespace icb {

constexpr int kConvAhead = 4;      // rows whose loads are in flight per thread

template <typename T, int TAPS>
__global__ void __launch_bounds__(256) short_conv_kernel(const ConvArgs<T> a, T* __restrict__ y, long long ldy, int rows,
                                                         int run, int keep) {
  constexpr int V = kVec<T>;
  const int per_row = a.C / V;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const long long at = idx / per_row * run;
  if (at >= rows) return;
  const int r0 = (int)at, r1 = min(rows, r0 + run);
  const int most = (TAPS > 0 ? TAPS : a.taps) - 1;
  ConvLane<T, TAPS> lane;
  lane.init(a, (int)(idx % per_row) * V);
  int before = rows_before(a.seqs, r0, most), slot = a.seqs[r0];
  lane.refill(a, r0, before, slot, a.pos[r0]);
  for (int g = r0; g < r1; g += kConvAhead) {
    uint4 x[kConvAhead];
    int s[kConvAhead];
#pragma unroll
    for (int i = 0; i < kConvAhead; ++i)
      if (g + i < r1) {
        x[i] = lane.fetch(a, g + i);
        s[i] = a.seqs[g + i];
      }
#pragma unroll
    for (int i = 0; i < kConvAhead; ++i) {
      const int r = g + i;
      if (r >= r1) break;
      if (r > r0) {
        if (s[i] == slot) {
          before = min(before + 1, most);
        } else {
          before = 0;
          slot = s[i];
          lane.refill(a, r, 0, slot, a.pos[r]);
        }
      }
      const int pos = TAPS > 0 && !keep ? 0 : a.pos[r];      // the register window does not ask
      float out[V];
      lane.row(a, x[i], r, before, slot, pos, out);
      store_row<T>(y + (size_t)r * ldy + lane.ch, out);
      if (keep) conv_keep<T>(a, r, before, slot, pos, lane.ch);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) conv_keep_kernel(const ConvArgs<T> a, const int* __restrict__ cu, int n) {
  const int per_row = a.C / kVec<T>;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int i = (int)(idx / per_row);
  if (i >= n) return;
  const int r = cu[i + 1] - 1;
  if (r < cu[i]) return;
  conv_keep<T>(a, r, min(r - cu[i], a.taps - 1), a.seqs[r], a.pos[r], (int)(idx % per_row) * kVec<T>);
}

template <typename T>
static int launch_conv(const ConvArgs<T>& a, T* y, long long ldy, const int* cu, int n, int rows, cudaStream_t st) {
  const int per_row = a.C / kVec<T>;
  if (y != nullptr) {
    const int run = cu == nullptr ? 1 : conv_run(rows, per_row, num_sms(), 2 * 256);
    const long long threads = (long long)((rows + run - 1) / run) * per_row;
    const int blocks = (int)((threads + 255) / 256);
    const int keep = cu == nullptr && a.taps > 1;     // every row is its sequence's only one: nobody else reads the state
    if (a.taps == 4) short_conv_kernel<T, 4><<<blocks, 256, 0, st>>>(a, y, ldy, rows, run, keep);
    else if (a.taps == 3) short_conv_kernel<T, 3><<<blocks, 256, 0, st>>>(a, y, ldy, rows, run, keep);
    else if (a.taps == 2) short_conv_kernel<T, 2><<<blocks, 256, 0, st>>>(a, y, ldy, rows, run, keep);
    else short_conv_kernel<T, 0><<<blocks, 256, 0, st>>>(a, y, ldy, rows, run, keep);
    int rc = check_launch("short_conv_kernel");
    if (rc) return rc;
  }
  if (cu != nullptr && a.taps > 1) {
    const long long threads = (long long)n * per_row;
    conv_keep_kernel<T><<<(int)((threads + 255) / 256), 256, 0, st>>>(a, cu, n);
    return check_launch("conv_keep_kernel");
  }
  return 0;
}

}  // namespace icb

using namespace icb;

// y[rows, pitch ldy] = silu(conv(x)) over C channels (a multiple of 8; pitches multiples of 8), and the carried inputs
// state[slots, taps - 1, C]. cu [n + 1] bounds the sequences' rows; null: one row per sequence. y == null: the state
// only (cu required). x, y, state: bf16 or fp32 (dtype); w [taps][C] and bias fp32.
ICB_API int icb_short_conv(const void* x, long long ldx, const float* w, const float* bias, void* state, const int* seqs,
                           const int* pos, const int* cu, int n, void* y, long long ldy, int rows, int C, int taps,
                           int dtype, void* stream) {
  if (rows <= 0 || C <= 0) return 0;
  if (C % 8 || ldx % 8 || ldy % 8 || taps < 1) return -2;
  if (y == nullptr && cu == nullptr) return -4;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (dtype == kBF16) {
    using T = __nv_bfloat16;
    ConvArgs<T> a{(const T*)x, ldx, w, bias, (T*)state, seqs, pos, C, taps};
    return launch_conv<T>(a, (T*)y, ldy, cu, n, rows, st);
  }
  if (dtype == kF32) {
    ConvArgs<float> a{(const float*)x, ldx, w, bias, (float*)state, seqs, pos, C, taps};
    return launch_conv<float>(a, (float*)y, ldy, cu, n, rows, st);
  }
  return -3;
}
