// Short causal convolution over time with silu, for rows of many sequences (see rows.cuh), and the update of the
// inputs that every sequence carries along.
#include "host_common.h"
#include "rows.cuh"

namespace icb {

template <typename T, int TAPS>
__global__ void __launch_bounds__(256) short_conv_kernel(const ConvArgs<T> a, T* __restrict__ y, long long ldy, int rows,
                                                         int run, int keep) {
  constexpr int V = kVec<T>;
  const int per_row = a.C / V;
  const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int r0 = (int)(idx / per_row) * run;
  if (r0 >= rows) return;
  const int ch = (int)(idx % per_row) * V;
  const int most = (TAPS > 0 ? TAPS : a.taps) - 1;
  ConvWeights<T, TAPS> k;
  load_conv_weights<T, TAPS>(a, ch, k);
  int before = rows_before(a.seqs, r0, most);
  const int r1 = min(rows, r0 + run);
  int slot = a.seqs[r0];
  for (int r = r0; r < r1; ++r) {
    if (r > r0) {
      const int s = a.seqs[r];
      before = s == slot ? min(before + 1, most) : 0;
      slot = s;
    }
    const int pos = a.pos[r];
    float out[V];
    conv_silu_row<T, TAPS>(a, k, r, before, slot, pos, ch, out);
    store_row<T>(y + (size_t)r * ldy + ch, out);
    if (keep) conv_keep<T>(a, r, before, slot, pos, ch);
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
    const int run = cu == nullptr ? 1 : conv_run(rows, per_row, num_sms());
    const long long threads = (long long)((rows + run - 1) / run) * per_row;
    const int blocks = (int)((threads + 255) / 256);
    const int keep = cu == nullptr && a.taps > 1;     // every row is its sequence's only one: nobody else reads the state
    if (a.taps == 4) short_conv_kernel<T, 4><<<blocks, 256, 0, st>>>(a, y, ldy, rows, run, keep);
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
