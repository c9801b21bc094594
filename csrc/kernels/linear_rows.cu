// bf16 linear layers of one to eight rows (decode): the weights are streamed once, y[M, N] = x[M, K] W[N, K]^T with fp32
// accumulation, fp32 / bf16 output or a SiLU(gate) * up epilogue. A warp owns two weight rows (a gate and its up row for
// SwiGLU) and, when there are too few rows to fill the machine, a slice of K; the slices of a block are added in a fixed
// order. The first weights are requested before the wait for the previous kernel. Weight rows from `split` on may have an input of
// their own: two products whose inputs come from the same step in one launch.
#include "../common/pk_common.cuh"

namespace {

using namespace pk;

enum { OUT_BF16 = 0, OUT_SWIGLU = 1, OUT_F32 = 2 };
constexpr int WARPS = 8;

struct RowsParams {
  const bf16* x;
  const bf16* x2;           // input of weight rows from `split` (even) on
  int split, ldx;
  const bf16* w;
  int N, K, epi, ksplit;    // ksplit: warps of a block that share a row pair (1, 2, 4, 8)
  void* y;
  int ldy;
};

__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

template <int M, int U>
__global__ void __launch_bounds__(32 * WARPS) linear_rows_kernel(const RowsParams p) {
  __shared__ float part[WARPS][2][M];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ks = p.ksplit, per_block = WARPS / ks;
  const int groups = p.epi == OUT_SWIGLU ? p.N / 2 : (p.N + 1) / 2;
  const int g = blockIdx.x * per_block + warp / ks, sl = warp % ks;
  const bool live = g < groups;
  const int n0 = p.epi == OUT_SWIGLU ? g : 2 * g;
  const int n1 = p.epi == OUT_SWIGLU ? g + groups : min(2 * g + 1, p.N - 1);
  const bf16* w0 = p.w + (size_t)(live ? n0 : 0) * p.K;
  const bf16* w1 = p.w + (size_t)(live ? n1 : 0) * p.K;
  const bf16* x = n0 < p.split ? p.x : p.x2;
  const int stride = 256 * ks;
  int k = sl * 256 + lane * 8;
  uint4 a[U], b[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    a[u] = b[u] = make_uint4(0, 0, 0, 0);
    if (live && k + u * stride < p.K) {
      a[u] = ld_stream_u4(w0 + k + u * stride);
      b[u] = ld_stream_u4(w1 + k + u * stride);
    }
  }
  pdl_trigger();
  pdl_wait();
  float acc0[M], acc1[M];
#pragma unroll
  for (int m = 0; m < M; ++m) acc0[m] = acc1[m] = 0.f;
  while (live && k < p.K) {
    const int kn = k + U * stride;
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int kk = k + u * stride;
      if (kk < p.K) {
        float fa[8], fb[8];
        unpack8(a[u], fa);
        unpack8(b[u], fb);
        // refill before the arithmetic: the next stretch is in flight meanwhile
        if (kk + U * stride < p.K) {
          a[u] = ld_stream_u4(w0 + kk + U * stride);
          b[u] = ld_stream_u4(w1 + kk + U * stride);
        }
#pragma unroll
        for (int m = 0; m < M; ++m) {
          float fx[8];
          unpack8(*reinterpret_cast<const uint4*>(x + (size_t)m * p.ldx + kk), fx);
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            acc0[m] = fmaf(fa[e], fx[e], acc0[m]);
            acc1[m] = fmaf(fb[e], fx[e], acc1[m]);
          }
        }
      }
    }
    k = kn;
  }
#pragma unroll
  for (int m = 0; m < M; ++m) {
    acc0[m] = warp_sum(acc0[m]);
    acc1[m] = warp_sum(acc1[m]);
  }
  if (ks > 1) {
    if (lane == 0) {
#pragma unroll
      for (int m = 0; m < M; ++m) {
        part[warp][0][m] = acc0[m];
        part[warp][1][m] = acc1[m];
      }
    }
    __syncthreads();
    if (sl == 0 && lane == 0) {
      for (int s = 1; s < ks; ++s)
#pragma unroll
        for (int m = 0; m < M; ++m) {
          acc0[m] += part[warp + s][0][m];
          acc1[m] += part[warp + s][1][m];
        }
    }
  }
  if (live && sl == 0 && lane == 0) {
#pragma unroll
    for (int m = 0; m < M; ++m) {
      if (p.epi == OUT_SWIGLU) {
        reinterpret_cast<bf16*>(p.y)[(size_t)m * p.ldy + g] = __float2bfloat16(silu(acc0[m]) * acc1[m]);
      } else if (p.epi == OUT_F32) {
        float* y = reinterpret_cast<float*>(p.y) + (size_t)m * p.ldy;
        y[n0] = acc0[m];
        if (2 * g + 1 < p.N) y[n1] = acc1[m];
      } else {
        bf16* y = reinterpret_cast<bf16*>(p.y) + (size_t)m * p.ldy;
        y[n0] = __float2bfloat16(acc0[m]);
        if (2 * g + 1 < p.N) y[n1] = __float2bfloat16(acc1[m]);
      }
    }
  }
}

}  // namespace

// As pk_linear_rows; x2 has the same stride and is the input of the weight rows from `split` (a multiple of 2) on.
PK_API int pk_linear_rows2(const void* x, const void* x2, int split, int ldx, const void* w, int M, int N, int K, int epi, void* y, int ldy, int sm_count,
                           cudaStream_t stream) {
  if (x2 == nullptr || ((uintptr_t)x2 & 15) != 0 || split < 0 || (split & 1) != 0 || (epi == OUT_SWIGLU && split < N)) return PK_ERR_BAD_ARG;
  if (M < 1 || M > 8 || N < 1 || K < 8 || (K & 7) != 0 || (ldx & 7) != 0 || ldx < K || epi < 0 || epi > 2) return PK_ERR_BAD_ARG;
  if (((uintptr_t)x & 15) != 0 || ((uintptr_t)w & 15) != 0 || (epi == OUT_SWIGLU && (N & 1) != 0)) return PK_ERR_BAD_ARG;
  if (ldy < (epi == OUT_SWIGLU ? N / 2 : N)) return PK_ERR_BAD_ARG;
  const int groups = epi == OUT_SWIGLU ? N / 2 : (N + 1) / 2;
  const int want = (sm_count > 0 ? sm_count : 148) * 16;      // warps that keep enough loads in flight
  int ks = 1;
  while (ks < WARPS && groups * ks < want && K >= 512 * ks * 2) ks *= 2;
  RowsParams p{(const pk::bf16*)x, (const pk::bf16*)x2, split, ldx, (const pk::bf16*)w, N, K, epi, ks, y, ldy};
  const dim3 grid((groups + WARPS / ks - 1) / (WARPS / ks)), block(32 * WARPS);
  switch (M) {
    case 1: PK_LAUNCH_PDL((linear_rows_kernel<1, 4>), grid, block, (size_t)0, stream, p); break;
    case 2: PK_LAUNCH_PDL((linear_rows_kernel<2, 4>), grid, block, (size_t)0, stream, p); break;
    case 3: PK_LAUNCH_PDL((linear_rows_kernel<3, 2>), grid, block, (size_t)0, stream, p); break;
    case 4: PK_LAUNCH_PDL((linear_rows_kernel<4, 2>), grid, block, (size_t)0, stream, p); break;
    case 5: PK_LAUNCH_PDL((linear_rows_kernel<5, 2>), grid, block, (size_t)0, stream, p); break;
    case 6: PK_LAUNCH_PDL((linear_rows_kernel<6, 2>), grid, block, (size_t)0, stream, p); break;
    case 7: PK_LAUNCH_PDL((linear_rows_kernel<7, 2>), grid, block, (size_t)0, stream, p); break;
    default: PK_LAUNCH_PDL((linear_rows_kernel<8, 2>), grid, block, (size_t)0, stream, p); break;
  }
  return PK_OK;
}

// x [M <= 8, K] bf16 rows (stride ldx, K and ldx multiples of 8, 16-byte aligned), W [N, K] bf16. epi 0 bf16, 1 SwiGLU (N / 2
// gate rows, then N / 2 up rows; bf16 out), 2 fp32.
PK_API int pk_linear_rows(const void* x, int ldx, const void* w, int M, int N, int K, int epi, void* y, int ldy, int sm_count, cudaStream_t stream) {
  return pk_linear_rows2(x, x, (N + 1) & ~1, ldx, w, M, N, K, epi, y, ldy, sm_count, stream);
}
