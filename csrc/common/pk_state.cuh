// Descriptor of recurrent mixers with an outer-product state (linear_state.cu, ssd.cu), plain data mirrored by the Python
// bindings; inputs of the state-space recurrence.
#pragma once
#include "pk_common.cuh"

// All pointers are device pointers; what the fields mean for which kind of recurrence is in linear_state.cu.
struct PkStateMixer {
  const float* proj;
  const float* bi;
  const float* bf;
  const float* a2;
  const float* a2b;
  float* S;
  float* N;
  float* Ms;
  float* o;
  float* nq;
  float* m;
  const double* freq;
  const float* pw;
  const float* cw;
  const float* cb;
  const float* dtb;
  const float* A;
  const float* skip;
  float* Cs;
  const float* low;
  int kind, ld, oq, ok, ov, og, oi, of, oa, H, D, V, rank, rot, groups, taps, odt;
  float qscale, cap, inv_tau;
};

namespace pk {

// The state space's convolved channels: x (H x V) | B (groups x D) | C (groups x D).
template <typename M>
__device__ __host__ __forceinline__ int ssd_channels(const M& mx) { return mx.H * mx.V + 2 * mx.groups * mx.D; }

// Input of the convolution `lag` tokens before the one at `row`, which is token `t` of its portion, at position pos: from the
// projection, or from the slot's ring [position modulo (taps - 1)][channel].
template <typename M>
__device__ __forceinline__ float conv_input(const M& mx, int slot, int row, int t, int pos, int lag, int ch) {
  if (lag > pos) return 0.f;
  const float* ring = mx.Cs + ((size_t)slot * (mx.taps - 1) + (pos - lag) % max(mx.taps - 1, 1)) * ssd_channels(mx) + ch;
  return *(lag <= t ? mx.proj + (size_t)(row - lag) * mx.ld + mx.ov + ch : ring);
}

__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }

// Convolution and SiLU of one channel; TAPS 0: any number of taps.
template <int TAPS, typename M>
__device__ __forceinline__ float conv_silu(const M& mx, int slot, int row, int t, int pos, int ch) {
  float y = mx.cb[ch];
  if (TAPS > 0) {
    constexpr int N = TAPS > 0 ? TAPS : 1;
    float x[N];
#pragma unroll
    for (int j = 0; j < N; ++j) x[j] = conv_input(mx, slot, row, t, pos, N - 1 - j, ch);
#pragma unroll
    for (int j = 0; j < N; ++j) y = fmaf(mx.cw[(size_t)ch * N + j], x[j], y);
  } else {
    for (int j = 0; j < mx.taps; ++j) y = fmaf(mx.cw[(size_t)ch * mx.taps + j], conv_input(mx, slot, row, t, pos, mx.taps - 1 - j, ch), y);
  }
  return silu_exact(y);
}

// Convolution and SiLU of one channel over `n` consecutive rows from `row` on (token `t` of its portion, at position pos).
template <int TAPS, typename M, typename Put>
__device__ __forceinline__ void conv_silu_rows(const M& mx, int slot, int row, int t, int pos, int n, int ch, Put put) {
  if (TAPS == 0) {
    for (int r = 0; r < n; ++r) put(r, conv_silu<0>(mx, slot, row + r, t + r, pos + r, ch));
    return;
  }
  constexpr int N = TAPS > 0 ? TAPS : 1, AHEAD = 8;
  float w[N], win[N];
#pragma unroll
  for (int j = 0; j < N; ++j) w[j] = mx.cw[(size_t)ch * N + j];
  const float b = mx.cb[ch];
  win[0] = 0.f;
#pragma unroll
  for (int j = 0; j + 1 < N; ++j) win[j + 1] = conv_input(mx, slot, row, t, pos, N - 1 - j, ch);
  const float* in = mx.proj + (size_t)row * mx.ld + mx.ov + ch;
  for (int r0 = 0; r0 < n; r0 += AHEAD) {
    float x[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) x[i] = r0 + i < n ? in[(size_t)(r0 + i) * mx.ld] : 0.f;
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
#pragma unroll
      for (int j = 0; j + 1 < N; ++j) win[j] = win[j + 1];
      win[N - 1] = x[i];
      float y = b;
#pragma unroll
      for (int j = 0; j < N; ++j) y = fmaf(w[j], win[j], y);
      if (r0 + i < n) put(r0 + i, silu_exact(y));
    }
  }
}

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// One warp, one head: step sizes of a chunk of 32 PER tokens (rows from `row` on, `len` of them real, the others with step 0) and
// the running log decay A dt, summed in double precision and kept as the sum of two floats. Lane l has tokens PER l ...
template <int PER, typename M>
__device__ __forceinline__ void ssd_decays(const M& mx, int row, int len, int h, int lane, float* dt_out, float2* g_out, float* total) {
  float dt[PER];
  double own = 0.0;
  const double a = (double)mx.A[h];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int r = PER * lane + i;
    dt[i] = r < len ? softplus(mx.proj[(size_t)(row + r) * mx.ld + mx.odt + h] + mx.dtb[h]) : 0.f;
    own += a * dt[i];
  }
  double run = own;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += v;
  }
  double g = run - own;
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    g += a * dt[i];
    const float hi = (float)g;
    g_out[PER * lane + i] = make_float2(hi, (float)(g - (double)hi));
    dt_out[PER * lane + i] = dt[i];
  }
  if (lane == 31) *total = (float)run;
}

}  // namespace pk
