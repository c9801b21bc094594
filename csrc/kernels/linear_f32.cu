// fp32 linear layers (no reduced-precision tensor mode): y[M, N] = x[M, K] W[N, K]^T with fp32 operands and fp32 FMA
// accumulation, optional SiLU(gate) * up epilogue. This is the 32-bit counterpart of the bf16 GEMM and matvec kernels for
// running a model entirely in fp32; up to eight rows stream the weights (one warp per output column), more rows use
// 64 x 64 tiles.
#include "../common/pk_common.cuh"

namespace {

using namespace pk;

struct LinParams {
  const float* x;
  int ldx;
  const float* w;     // [N, K]; SwiGLU: N / 2 gate rows, then N / 2 up rows
  int M, N, K, swiglu;
  float* y;
  int ldy;
};

__device__ __forceinline__ float silu_exact(float z) { return z / (1.f + expf(-z)); }

template <int MR>
__global__ void __launch_bounds__(256) linear_f32_rows_kernel(const LinParams p) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ncol = p.swiglu ? p.N / 2 : p.N;
  const int n = blockIdx.x * 8 + warp;
  if (n >= ncol) return;
  float a[MR], b[MR];
#pragma unroll
  for (int m = 0; m < MR; ++m) a[m] = b[m] = 0.f;
  const float* w0 = p.w + (size_t)n * p.K;
  const float* w1 = p.w + (size_t)(n + ncol) * p.K;
  for (int k = lane; k < p.K; k += 32) {
    const float wa = w0[k], wb = p.swiglu ? w1[k] : 0.f;
#pragma unroll
    for (int m = 0; m < MR; ++m) {
      if (m < p.M) {
        const float xv = p.x[(size_t)m * p.ldx + k];
        a[m] = fmaf(xv, wa, a[m]);
        if (p.swiglu) b[m] = fmaf(xv, wb, b[m]);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MR; ++m) {
    a[m] = warp_sum(a[m]);
    if (p.swiglu) b[m] = warp_sum(b[m]);
    if (lane == 0 && m < p.M) p.y[(size_t)m * p.ldy + n] = p.swiglu ? silu_exact(a[m]) * b[m] : a[m];
  }
}

constexpr int TB = 64, TK = 16;

__global__ void __launch_bounds__(256) linear_f32_tile_kernel(const LinParams p) {
  __shared__ float xs[TK][TB + 4], ws[TK][TB + 4], us[TK][TB + 4];
  const int m0 = blockIdx.y * TB, n0 = blockIdx.x * TB, tid = threadIdx.x;
  const int ncol = p.swiglu ? p.N / 2 : p.N;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4], up[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = up[i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += TK) {
    for (int i = tid; i < TB * TK; i += 256) {
      const int r = i / TK, k = i - r * TK;
      const bool kin = k0 + k < p.K;
      xs[k][r] = kin && m0 + r < p.M ? p.x[(size_t)(m0 + r) * p.ldx + k0 + k] : 0.f;
      ws[k][r] = kin && n0 + r < ncol ? p.w[(size_t)(n0 + r) * p.K + k0 + k] : 0.f;
      if (p.swiglu) us[k][r] = kin && n0 + r < ncol ? p.w[(size_t)(ncol + n0 + r) * p.K + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float4 xa = *reinterpret_cast<const float4*>(&xs[k][ty * 4]);
      const float4 wa = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float xv[4] = {xa.x, xa.y, xa.z, xa.w}, wv[4] = {wa.x, wa.y, wa.z, wa.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], wv[j], acc[i][j]);
      if (p.swiglu) {
        const float4 ua = *reinterpret_cast<const float4*>(&us[k][tx * 4]);
        const float uv[4] = {ua.x, ua.y, ua.z, ua.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) up[i][j] = fmaf(xv[i], uv[j], up[i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n < ncol) p.y[(size_t)m * p.ldy + n] = p.swiglu ? silu_exact(acc[i][j]) * up[i][j] : acc[i][j];
    }
  }
}

}  // namespace

PK_API int pk_linear_f32(const float* x, int ldx, const float* w, int M, int N, int K, int swiglu, float* y, int ldy, cudaStream_t stream) {
  if (M < 1 || N < 1 || K < 1 || ldx < K || (swiglu && (N & 1) != 0)) return PK_ERR_BAD_ARG;
  const int ncol = swiglu ? N / 2 : N;
  if (ldy < ncol) return PK_ERR_BAD_ARG;
  LinParams p{x, ldx, w, M, N, K, swiglu, y, ldy};
  if (M <= 8) {
    const int g = (ncol + 7) / 8;
    if (M == 1) linear_f32_rows_kernel<1><<<g, 256, 0, stream>>>(p);
    else if (M <= 4) linear_f32_rows_kernel<4><<<g, 256, 0, stream>>>(p);
    else linear_f32_rows_kernel<8><<<g, 256, 0, stream>>>(p);
  } else {
    linear_f32_tile_kernel<<<dim3((ncol + TB - 1) / TB, (M + TB - 1) / TB), 256, 0, stream>>>(p);
  }
  PK_CHECK_LAUNCH();
  return PK_OK;
}
