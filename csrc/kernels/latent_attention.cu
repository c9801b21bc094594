// Latent attention over a paged cache: a cached row is [latent c (rms-normed) | rotated key part | zero padding], shared by
// all heads; per head the unrotated key is W_uk c and the value W_uv c. Causal with an optional sliding window and an
// optional learned sink per head (a score without key and value that counts once in the denominator). The rotated part may be
// empty; queries may come from a latent of their own (normed by prep, expanded by a product behind it); the heads' outputs may be
// multiplied with a sigmoid gate, element by element.
//
//   prep     per row: norm of the latent, rotation (rotate-half, any frequency table) of key part and queries, cache
//            append, queries for the tensor-core kernel
//   gather   cached rows of the positions a long portion can see -> contiguous rows (input of the key / value GEMM)
//   absorb   q~ = W_uk^T q per head (few rows: scores are taken on the latent, keys are never expanded)
//   rows     split-context attention of single rows over the cache, eight heads per block, online softmax in fp32
//   merge    sum of the splits, with the sink in the denominator
//   out      W_uv per head
// Scores, weights and accumulators are fp32 in all of them; the cache and the weights are bf16 or (fp32 mode) fp32.
#include "../common/pk_rotary.cuh"

namespace {

using namespace pk;

constexpr int kPage = 64;    // tokens per page
constexpr int HB = 8;        // heads of a rows block
constexpr int TK = 32;       // cached rows of a tile

struct Paged {
  void* cache;            // [pages, 64, row]
  const int* table;       // [slots, table_ld] page of every 64 positions
  int table_ld, row;      // row = elements per cached position
};

__device__ __forceinline__ size_t cache_row(const Paged& c, int slot, int pos) {
  return ((size_t)c.table[(size_t)slot * c.table_ld + pos / kPage] * kPage + pos % kPage) * c.row;
}

template <typename T>
__device__ __forceinline__ float to_f(T v) { return (float)v; }
template <>
__device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }

struct PrepParams {
  const float* proj;      // [rows, ld]: q (H x [D | R]) at oq, latent | key part at oc
  int ld, oq, oc, H, D, R, K;
  const float* c_norm;    // [K] plain weight
  float eps;
  const double* freq;     // [R / 2]
  float mag;              // factor on cos and sin
  const int* pos;
  const int* slot;
  Paged c;
  float* qx;              // [rows, H, row]: columns K .. K + R <- rotated query, the padding <- 0 (null: skip)
  bf16* qf;               // [rows, H, qf_ld]: whole rotated query, padding <- 0 (null: skip)
  int qf_ld;
  // queries from a latent: QK columns at oq -> normed rows for the product that expands them
  int QK;                 // 0: the queries themselves are in proj
  const float* q_norm;    // [QK]
  void* ql;               // [rows, ql_ld], the cache's type, padding <- 0
  int ql_ld;
};

// dst[0 .. n) = normed src times w, zeros up to `padded`. Whole block.
template <typename T>
__device__ __forceinline__ void norm_row(const float* src, int n, const float* w, float eps, T* dst, int padded, float* scratch) {
  float ss = 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) ss = fmaf(src[i], src[i], ss);
  const float r = 1.f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  for (int i = threadIdx.x; i < padded; i += blockDim.x) dst[i] = (T)(i < n ? src[i] * r * w[i] : 0.f);
}

// Block (row, group of eight heads), one warp per head; the first group also writes the cache row. Queries from a latent: the second
// block of a row norms it.
template <typename CT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const PrepParams p) {
  pdl_trigger();
  extern __shared__ float sm[];      // cos, sin [R / 2] each
  __shared__ float scratch[33];
  const int t = blockIdx.x, tid = threadIdx.x, half = p.R / 2;
  const int warp = tid >> 5, lane = tid & 31;
  pdl_wait();
  const float* pr = p.proj + (size_t)t * p.ld;
  if (p.QK > 0 && blockIdx.y == 1) {
    norm_row<CT>(pr + p.oq, p.QK, p.q_norm, p.eps, reinterpret_cast<CT*>(p.ql) + (size_t)t * p.ql_ld, p.ql_ld, scratch);
    return;
  }
  const int pos = p.pos[t];
  float* cs = sm;
  float* sn = sm + half;
  for (int i = tid; i < half; i += 256) {
    float s, c;
    rotary_sincos(p.freq[i], pos, s, c);
    cs[i] = c * p.mag;
    sn[i] = s * p.mag;
  }
  if (blockIdx.y == 0) {
    float ss = 0.f;
    for (int i = tid; i < p.K; i += 256) {
      const float v = pr[p.oc + i];
      ss = fmaf(v, v, ss);
    }
    const float r = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.K + p.eps);   // also orders cs / sn
    CT* dst = reinterpret_cast<CT*>(p.c.cache) + cache_row(p.c, p.slot[t], pos);
    for (int i = tid; i < p.c.row; i += 256) {
      float v = 0.f;
      if (i < p.K) v = pr[p.oc + i] * r * p.c_norm[i];
      else if (i < p.K + p.R) {
        const int j = i - p.K;
        const float* kr = pr + p.oc + p.K;
        v = j < half ? kr[j] * cs[j] - kr[j + half] * sn[j] : kr[j] * cs[j - half] + kr[j - half] * sn[j - half];
      }
      dst[i] = (CT)v;
    }
  } else {
    __syncthreads();
  }
  const int h = blockIdx.y * 8 + warp;
  if (h >= p.H || p.QK > 0) return;
  const float* q = pr + p.oq + h * (p.D + p.R);
  const float* qr = q + p.D;
  auto rotated = [&](int j) {
    return j < half ? qr[j] * cs[j] - qr[j + half] * sn[j] : qr[j] * cs[j - half] + qr[j - half] * sn[j - half];
  };
  if (p.qx) {
    float* dst = p.qx + ((size_t)t * p.H + h) * p.c.row + p.K;
    for (int j = lane; j < p.c.row - p.K; j += 32) dst[j] = j < p.R ? rotated(j) : 0.f;
  }
  if (p.qf) {
    bf16* dst = p.qf + ((size_t)t * p.H + h) * p.qf_ld;
    for (int j = lane; j < p.qf_ld; j += 32) dst[j] = __float2bfloat16(j < p.D ? q[j] : j < p.D + p.R ? rotated(j - p.D) : 0.f);
  }
}

// seqs {first row, tokens, slot, first position}; gather {first gathered row, first gathered position} per sequence.
__global__ void __launch_bounds__(128) latent_gather_kernel(const Paged c, const int4* seqs, const int2* gather, bf16* out) {
  const int4 sq = seqs[blockIdx.y];
  const int2 g = gather[blockIdx.y];
  const int n = sq.w + sq.y - g.y, vec = c.row / 8;
  const int per = 128 / 32;
  for (int i = blockIdx.x * per + (threadIdx.x >> 5); i < n; i += gridDim.x * per) {
    const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(c.cache) + cache_row(c, sq.z, g.y + i));
    uint4* dst = reinterpret_cast<uint4*>(out + (size_t)(g.x + i) * c.row);
    for (int v = threadIdx.x & 31; v < vec; v += 32) dst[v] = src[v];
  }
}

// qx[row, h, 0 .. K) = W_uk[h]^T q[h], zeros up to K_pad (what lies behind belongs to prep). Block: 128 latent columns of one head,
// up to 8 rows, 4 groups over the head dim.
template <typename WT>
__global__ void __launch_bounds__(512) latent_absorb_kernel(const float* proj, int ld, int oq, int H, int D, int R, int K, int K_pad, const WT* uk,
                                                           const int* rows, int nrows, float* qx, int row) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];          // q [8][D], partial sums [4][8][128]
  float* qs = sm;
  float* red = sm + 8 * D;
  const int h = blockIdx.x, k = blockIdx.y * 128 + (threadIdx.x & 127), grp = threadIdx.x >> 7;
  const int r0 = blockIdx.z * 8, nr = min(8, nrows - r0);
  for (int i = threadIdx.x; i < 8 * D; i += 512) {
    const int r = i / D, d = i - r * D;
    qs[i] = r < nr ? proj[(size_t)rows[r0 + r] * ld + oq + h * (D + R) + d] : 0.f;
  }
  __syncthreads();
  float acc[8];
#pragma unroll
  for (int r = 0; r < 8; ++r) acc[r] = 0.f;
  if (k < K) {
    const WT* w = uk + (size_t)h * D * K + k;
#pragma unroll 16
    for (int d = grp; d < D; d += 4) {
      const float wv = to_f<WT>(w[(size_t)d * K]);
#pragma unroll
      for (int r = 0; r < 8; ++r) acc[r] = fmaf(wv, qs[r * D + d], acc[r]);
    }
  }
#pragma unroll
  for (int r = 0; r < 8; ++r) red[(grp * 8 + r) * 128 + (threadIdx.x & 127)] = acc[r];
  __syncthreads();
  for (int i = threadIdx.x; i < nr * 128; i += 512) {
    const int r = i >> 7, c = i & 127;
    if (blockIdx.y * 128 + c < K_pad)      // columns behind K have summed nothing
      qx[((size_t)rows[r0 + r] * H + h) * row + blockIdx.y * 128 + c] =
          red[r * 128 + c] + red[(8 + r) * 128 + c] + red[(16 + r) * 128 + c] + red[(24 + r) * 128 + c];
  }
}

struct RowsParams {
  const float* qx;        // [rows, H, row]
  const int* rows;        // rows of the step that are attended here
  const int* pos;
  const int* slot;
  Paged c;
  int H, K, window, nsplit;
  float scale;
  float* part_o;          // [listed rows, nsplit, H, K]
  float* part_ml;         // [listed rows, nsplit, H, 2]
};

// One block: one row, HB heads, one split of its visible positions. Warp w owns head w's scores (lane = cached row of the
// tile); for the weighted sum every thread owns CP pairs of latent columns for all HB heads.
template <typename CT, int CP>
__global__ void __launch_bounds__(32 * HB) latent_rows_kernel(const RowsParams p) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smraw[];
  constexpr int VE = 16 / sizeof(CT);                   // elements of a 16-byte access
  const int row = p.c.row, kld = row + VE;              // padded tile row: consecutive rows start four banks apart
  float* qs = reinterpret_cast<float*>(smraw);          // [HB][row]
  CT* ks = reinterpret_cast<CT*>(qs + HB * row);        // [TK][kld]
  float* ps = reinterpret_cast<float*>(ks + TK * kld);  // [TK][HB]
  float* al = ps + TK * HB;                             // [HB]
  const int li = blockIdx.x, h0 = blockIdx.y * HB, sp = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;
  const int t = p.rows[li], pos = p.pos[t], slot = p.slot[t];
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int n = pos + 1 - first;
  const int per = ((n + p.nsplit - 1) / p.nsplit + TK - 1) / TK * TK;
  const int s0 = first + sp * per, s1 = min(pos + 1, s0 + per);
  const int nh = min(HB, p.H - h0);
  {
    const float4* src = reinterpret_cast<const float4*>(p.qx + ((size_t)t * p.H + h0) * row);
#pragma unroll 5
    for (int i = tid; i < HB * row / 4; i += 32 * HB)
      reinterpret_cast<float4*>(qs)[i] = i < nh * row / 4 ? src[i] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float m = -INFINITY, l = 0.f;
  float acc[CP][2][HB];
#pragma unroll
  for (int a = 0; a < CP; ++a)
#pragma unroll
    for (int h = 0; h < HB; ++h) acc[a][0][h] = acc[a][1][h] = 0.f;
  const int vec = row / VE;
  for (int k0 = s0; k0 < s1; k0 += TK) {
    const int nk = min(TK, s1 - k0);
    __syncthreads();
    // four rows per warp; their addresses first, so that all loads of a column of lanes are in flight together
    constexpr int RW = TK / HB;
    const CT* src[RW];
#pragma unroll
    for (int j = 0; j < RW; ++j) {
      const int r = warp + j * HB;
      src[j] = reinterpret_cast<const CT*>(p.c.cache) + cache_row(p.c, slot, k0 + min(r, nk - 1));
    }
#pragma unroll 3
    for (int v = lane; v < vec; v += 32) {
      uint4 x[RW];
#pragma unroll
      for (int j = 0; j < RW; ++j) x[j] = *reinterpret_cast<const uint4*>(src[j] + v * VE);
#pragma unroll
      for (int j = 0; j < RW; ++j) *reinterpret_cast<uint4*>(ks + (warp + j * HB) * kld + v * VE) = x[j];
    }
    __syncthreads();
    float s4[4] = {0.f, 0.f, 0.f, 0.f};
    {
      const CT* kr = ks + lane * kld;
      const float* q = qs + warp * row;
#pragma unroll 4
      for (int v = 0; v < row; v += VE) {
        const uint4 raw = *reinterpret_cast<const uint4*>(kr + v);
        const CT* ke = reinterpret_cast<const CT*>(&raw);
#pragma unroll
        for (int e = 0; e < VE; ++e) s4[e & 3] = fmaf(to_f<CT>(ke[e]), q[v + e], s4[e & 3]);
      }
    }
    const float s = lane < nk ? ((s4[0] + s4[1]) + (s4[2] + s4[3])) * p.scale : -INFINITY;
    const float mn = fmaxf(m, warp_max(s));
    const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
    const float e = lane < nk ? expf(s - mn) : 0.f;
    l = l * alpha + warp_sum(e);
    m = mn;
    ps[lane * HB + warp] = e;
    if (lane == 0) al[warp] = alpha;
    __syncthreads();
    float a8[HB];
#pragma unroll
    for (int h = 0; h < HB; ++h) a8[h] = al[h];
#pragma unroll
    for (int a = 0; a < CP; ++a)
#pragma unroll
      for (int h = 0; h < HB; ++h) {
        acc[a][0][h] *= a8[h];
        acc[a][1][h] *= a8[h];
      }
    for (int r = 0; r < nk; ++r) {
      const float4 p0 = *reinterpret_cast<const float4*>(ps + r * HB), p1 = *reinterpret_cast<const float4*>(ps + r * HB + 4);
      const float pv[HB] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
#pragma unroll
      for (int a = 0; a < CP; ++a) {
        const int c = (a * 32 * HB + tid) * 2;
        if (c < row) {
          const float x0 = to_f<CT>(ks[r * kld + c]), x1 = to_f<CT>(ks[r * kld + c + 1]);
#pragma unroll
          for (int h = 0; h < HB; ++h) {
            acc[a][0][h] = fmaf(pv[h], x0, acc[a][0][h]);
            acc[a][1][h] = fmaf(pv[h], x1, acc[a][1][h]);
          }
        }
      }
    }
  }
  const size_t base = ((size_t)li * p.nsplit + sp) * p.H + h0;
  if (lane == 0 && warp < nh) {
    p.part_ml[(base + warp) * 2] = m;
    p.part_ml[(base + warp) * 2 + 1] = l;
  }
#pragma unroll
  for (int a = 0; a < CP; ++a) {
    const int c = (a * 32 * HB + tid) * 2;
#pragma unroll
    for (int h = 0; h < HB; ++h)
      if (h < nh) {
        if (c < p.K) p.part_o[(base + h) * p.K + c] = acc[a][0][h];
        if (c + 1 < p.K) p.part_o[(base + h) * p.K + c + 1] = acc[a][1][h];
      }
  }
}

struct OutParams {
  const float* part_o;    // merged: split 0
  int nsplit, H, K, V;
  const int* rows;
  int nrows;
  void* out;              // [rows of the step, ldo]
  int ldo;
  const float* gate;      // [rows of the step, ldg] logits of the gate, head h at h V (null: none)
  int ldg;
};

// o~[row, h, k] = sum over the splits, divided by the whole denominator (sink included). Written over split 0.
__global__ void __launch_bounds__(128) latent_merge_kernel(float* part_o, const float* part_ml, int nsplit, int H, int K, const float* sink) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float ws[];       // [nsplit]
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const float* ml = part_ml + ((size_t)r * nsplit * H + h) * 2;
  if (tid < 32) {
    float mx = sink ? sink[h] : -INFINITY;
    for (int s = lane; s < nsplit; s += 32) mx = fmaxf(mx, ml[(size_t)s * H * 2]);
    mx = warp_max(mx);
    float den = 0.f;
    for (int s = lane; s < nsplit; s += 32) {
      const float m = ml[(size_t)s * H * 2];
      const float e = m == -INFINITY ? 0.f : expf(m - mx);
      ws[s] = e;
      den += e * ml[(size_t)s * H * 2 + 1];
    }
    den = warp_sum(den) + (sink ? expf(sink[h] - mx) : 0.f);
    __syncwarp();
    for (int s = lane; s < nsplit; s += 32) ws[s] /= den;
  }
  __syncthreads();
  const int k = blockIdx.z * 128 + tid;
  if (k >= K) return;
  float* o = part_o + ((size_t)r * nsplit * H + h) * K + k;
  float a = 0.f;
  // an empty split holds zeros: every term is finite
#pragma unroll 8
  for (int s = 0; s < nsplit; ++s) a = fmaf(ws[s], o[(size_t)s * H * K], a);
  *o = a;
}

// out[row, h * V + v] = W_uv[h, v] . o~[row, h] for up to 8 rows of one head and 16 values.
template <typename WT, typename OutT>
__global__ void __launch_bounds__(256) latent_out_kernel(const OutParams p, const WT* uv) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float os[];       // o~ [8][K]
  const int h = blockIdx.x, r0 = blockIdx.y * 8, nr = min(8, p.nrows - r0), tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;
  for (int i = tid; i < nr * p.K; i += 256) {
    const int r = i / p.K, k = i - r * p.K;
    os[i] = p.part_o[((size_t)(r0 + r) * p.nsplit * p.H + h) * p.K + k];
  }
  __syncthreads();
  OutT* out = reinterpret_cast<OutT*>(p.out);
  for (int v = blockIdx.z * 16 + warp; v < min(p.V, (int)blockIdx.z * 16 + 16); v += 8) {
    const WT* w = uv + ((size_t)h * p.V + v) * p.K;
    float acc[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) acc[r] = 0.f;
#pragma unroll 8
    for (int k = lane; k < p.K; k += 32) {
      const float wv = to_f<WT>(w[k]);
#pragma unroll
      for (int r = 0; r < 8; ++r)
        if (r < nr) acc[r] = fmaf(wv, os[r * p.K + k], acc[r]);
    }
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      if (r >= nr) break;
      float s = warp_sum(acc[r]);
      if (lane == 0) {
        const size_t row = p.rows[r0 + r];
        if (p.gate) s /= 1.f + expf(-p.gate[row * p.ldg + h * p.V + v]);
        out[row * p.ldo + h * p.V + v] = (OutT)s;
      }
    }
  }
  if (h == p.H - 1 && blockIdx.z == 0)
    for (int i = tid; i < nr * (p.ldo - p.H * p.V); i += 256) {
      const int pad = p.ldo - p.H * p.V, r = i / pad;
      out[(size_t)p.rows[r0 + r] * p.ldo + p.H * p.V + (i - r * pad)] = (OutT)0.f;
    }
}

template <typename F>
int max_smem(F* fn, PkDeviceOnce& once, size_t smem) {
  if (PkDeviceOnceGuard g{once}; g.needed()) {
    if (cudaFuncSetAttribute((const void*)fn, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    g.done();
  }
  return smem <= 227 * 1024 ? PK_OK : PK_ERR_UNSUPPORTED;
}

template <typename CT, int CP>
int launch_rows(const RowsParams& p, int nrows, size_t smem, cudaStream_t stream) {
  static PkDeviceOnce once;
  const int rc = max_smem(latent_rows_kernel<CT, CP>, once, smem);
  if (rc != PK_OK) return rc;
  PK_LAUNCH_PDL((latent_rows_kernel<CT, CP>), dim3(nrows, (p.H + HB - 1) / HB, p.nsplit), dim3(32 * HB), smem, stream, p);
  return PK_OK;
}

}  // namespace

// See PrepParams. row (elements per cached position) is a multiple of 8 and at least K + R; R even. QK > 0: no rotated part, qx and
// qf are not written (the expanded queries are another product's output).
PK_API int pk_latent_prep(const float* proj, int ld, int oq, int oc, int M, int H, int D, int R, int K, const float* c_norm, float eps,
                          const double* freq, float mag, const int* pos, const int* slot, void* cache, const int* table, int table_ld,
                          int row, int cache_f32, float* qx, void* qf, int qf_ld, int QK, const float* q_norm, void* ql, int ql_ld, cudaStream_t stream) {
  if (M < 1 || H < 1 || D < 1 || R < 0 || (R & 1) != 0 || K < 1 || row < K + R || (row & 7) != 0 || cache == nullptr || table == nullptr) return PK_ERR_BAD_ARG;
  if (qf != nullptr && qf_ld < D + R) return PK_ERR_BAD_ARG;
  if (QK < 0 || (QK > 0 && (q_norm == nullptr || ql == nullptr || ql_ld < QK || R != 0))) return PK_ERR_BAD_ARG;
  PrepParams p{proj, ld, oq, oc, H, D, R, K, c_norm, eps, freq, mag, pos, slot, Paged{cache, table, table_ld, row}, qx, (pk::bf16*)qf, qf_ld, QK, q_norm, ql, ql_ld};
  const size_t smem = (size_t)(R + 2) * sizeof(float);
  const dim3 grid(M, QK > 0 ? 2 : (qx != nullptr || qf != nullptr) ? (H + 7) / 8 : 1);
  if (cache_f32) PK_LAUNCH_PDL(latent_prep_kernel<float>, grid, dim3(256), smem, stream, p);
  else PK_LAUNCH_PDL(latent_prep_kernel<pk::bf16>, grid, dim3(256), smem, stream, p);
  return PK_OK;
}

// bf16 cache rows of the positions [gather[s].y, end of portion s) -> out rows gather[s].x ...; max_rows = longest range.
PK_API int pk_latent_gather(const void* cache, const int* table, int table_ld, int row, const void* seqs, const void* gather, int nseq,
                            int max_rows, void* out, cudaStream_t stream) {
  if (nseq < 1 || max_rows < 1 || (row & 7) != 0 || ((uintptr_t)out & 15) != 0) return PK_ERR_BAD_ARG;
  const int blocks = (max_rows + 3) / 4;
  latent_gather_kernel<<<dim3(blocks < 592 ? blocks : 592, nseq), 128, 0, stream>>>(Paged{(void*)cache, table, table_ld, row}, (const int4*)seqs,
                                                                                 (const int2*)gather, (pk::bf16*)out);
  PK_CHECK_LAUNCH();
  return PK_OK;
}

// rows [nrows] of the step: qx columns 0 .. K_pad of their heads; R: what lies between the heads' D query columns.
PK_API int pk_latent_absorb(const float* proj, int ld, int oq, int H, int D, int R, int K, const void* uk, int w_f32, const int* rows, int nrows,
                            float* qx, int row, int K_pad, cudaStream_t stream) {
  if (nrows < 1 || H < 1 || D < 1 || K < 1 || K_pad < K || row < K_pad || qx == nullptr || rows == nullptr) return PK_ERR_BAD_ARG;
  const size_t smem = (size_t)(8 * D + 4 * 8 * 128) * sizeof(float);
  if (smem > 48 * 1024) return PK_ERR_UNSUPPORTED;
  const dim3 grid(H, (K_pad + 127) / 128, (nrows + 7) / 8);
  if (w_f32) PK_LAUNCH_PDL(latent_absorb_kernel<float>, grid, dim3(512), smem, stream, proj, ld, oq, H, D, R, K, K_pad, (const float*)uk, rows, nrows, qx, row);
  else PK_LAUNCH_PDL(latent_absorb_kernel<pk::bf16>, grid, dim3(512), smem, stream, proj, ld, oq, H, D, R, K, K_pad, (const pk::bf16*)uk, rows, nrows, qx, row);
  return PK_OK;
}

// window <= 0: full causal attention. part_o [nrows, nsplit, H, K] and part_ml [nrows, nsplit, H, 2] floats.
PK_API int pk_latent_rows(const float* qx, const int* rows, int nrows, const int* pos, const int* slot, const void* cache, const int* table,
                          int table_ld, int row, int cache_f32, int H, int K, int window, float scale, int nsplit, float* part_o,
                          float* part_ml, cudaStream_t stream) {
  if (nrows < 1 || H < 1 || K < 1 || nsplit < 1 || nsplit > 1024 || row < K || (row & 7) != 0 || part_o == nullptr || part_ml == nullptr) return PK_ERR_BAD_ARG;
  RowsParams p{qx, rows, pos, slot, Paged{(void*)cache, table, table_ld, row}, H, K, window, nsplit, scale, part_o, part_ml};
  const int es = cache_f32 ? 4 : 2;
  const size_t smem = (size_t)HB * row * 4 + (size_t)TK * (row + 16 / es) * es + (size_t)(TK * HB + HB) * 4;
  const int pairs = (row / 2 + 32 * HB - 1) / (32 * HB);
  if (cache_f32) {
    if (pairs <= 1) return launch_rows<float, 1>(p, nrows, smem, stream);
    if (pairs <= 2) return launch_rows<float, 2>(p, nrows, smem, stream);
    if (pairs <= 4) return launch_rows<float, 4>(p, nrows, smem, stream);
  } else {
    if (pairs <= 1) return launch_rows<pk::bf16, 1>(p, nrows, smem, stream);
    if (pairs <= 2) return launch_rows<pk::bf16, 2>(p, nrows, smem, stream);
    if (pairs <= 4) return launch_rows<pk::bf16, 4>(p, nrows, smem, stream);
  }
  return PK_ERR_UNSUPPORTED;
}

// Merge of the splits (in place), then W_uv and the gate. sink [H], gate [rows of the step, ldg] or null.
PK_API int pk_latent_out(float* part_o, const float* part_ml, int nsplit, int H, int K, int V, const float* sink, const int* rows, int nrows,
                         const void* uv, int f32, void* out, int ldo, const float* gate, int ldg, cudaStream_t stream) {
  if ((gate != nullptr && ldg < H * V) || nrows < 1 || nsplit < 1 || H < 1 || K < 1 || V < 1 || ldo < H * V) return PK_ERR_BAD_ARG;
  PK_LAUNCH_PDL(latent_merge_kernel, dim3(nrows, H, (K + 127) / 128), dim3(128), (size_t)nsplit * sizeof(float), stream, part_o, part_ml, nsplit, H, K, sink);
  OutParams p{part_o, nsplit, H, K, V, rows, nrows, out, ldo, gate, ldg};
  const size_t smem = (size_t)8 * K * sizeof(float);
  const dim3 grid(H, (nrows + 7) / 8, (V + 15) / 16);
  if (f32) {
    static PkDeviceOnce once;
    const int rc = max_smem(latent_out_kernel<float, float>, once, smem);
    if (rc != PK_OK) return rc;
    PK_LAUNCH_PDL((latent_out_kernel<float, float>), grid, dim3(256), smem, stream, p, (const float*)uv);
  } else {
    static PkDeviceOnce once;
    const int rc = max_smem(latent_out_kernel<pk::bf16, pk::bf16>, once, smem);
    if (rc != PK_OK) return rc;
    PK_LAUNCH_PDL((latent_out_kernel<pk::bf16, pk::bf16>), grid, dim3(256), smem, stream, p, (const pk::bf16*)uv);
  }
  return PK_OK;
}
