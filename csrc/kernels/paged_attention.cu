// Grouped-query attention over a paged cache, with the choices of its design as parameters: norms of queries and keys, rotation
// of a leading part of them (pairs half a width apart, or neighbours), values mixed with those of an earlier layer, full causal /
// sliding-window / chunked visibility, capped scores, a sink in the softmax, one softmax map per head or two over the same
// values whose difference a1 - lambda a2 is the head's output, an optional norm of every head's output, a gate per head.
//
//   prep    per row: norm, rotation, cache append, queries for the row kernel (fp32) and the tensor-core kernel (bf16)
//   rows    split-context attention of single rows: up to eight query vectors of one key head per block, fp32
//   merge   sum of the splits, difference of the maps, head norm
// Long portions of bf16 models run their attention in paged_prefill.cu.
#include "../common/pk_paged.h"
#include "../common/pk_rotary.cuh"

namespace {

using namespace pk;

constexpr int kPage = 64;    // positions per page
constexpr int QB = 8;        // query vectors of a rows block (one warp each for the scores)
constexpr int TK = 32;       // cached rows of a tile

typedef PkPagedAttention Attn;

__device__ __forceinline__ size_t cache_row(const Attn& a, int slot, int pos) {
  return ((size_t)a.table[(size_t)slot * a.table_ld + pos / kPage] * kPage + pos % kPage) * a.row;
}

__device__ __forceinline__ int first_visible(const Attn& a, int pos) {
  int f = 0;
  if (a.window > 0) f = max(f, pos - a.window + 1);
  if (a.chunk > 0) f = max(f, pos / a.chunk * a.chunk);
  return f;
}

template <typename T>
__device__ __forceinline__ float to_f(T v) { return (float)v; }
template <>
__device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }

// Block (row, share of the row's vectors), up to NPW vectors per warp, dealt out in turn: H x maps queries, G x maps keys, G
// values. The first pair of elements that a lane owns of every vector is on its way while the angles are computed.
template <typename CT, int NPW>
__global__ void __launch_bounds__(256) paged_prep_kernel(const Attn a) {
  pdl_trigger();
  extern __shared__ float sm[];      // cos, sin [R / 2] each
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, half = a.R / 2;
  const int nq = a.H * a.maps, nk = a.G * a.maps, total = nq + nk + a.G;
  const int v0 = blockIdx.y * 8 + warp, step = gridDim.y * 8;
  pdl_wait();
  const float* pr = a.proj + (size_t)t * a.ld;
  const int pos = a.pos[t];
  auto source = [&](int v) { return v < nq ? pr + a.oq + v * a.D : v < nq + nk ? pr + a.ok + (v - nq) * a.D : pr + a.ov + (v - nq - nk) * a.V; };
  // pair i of a query or key while it turns, then single elements
  const int pa = a.neighbours ? 2 : 1, pb = a.neighbours ? 1 : half;      // pair i: (i * pa, i * pa + pb)
  float x0[NPW], y0[NPW];
#pragma unroll
  for (int j = 0; j < NPW; ++j) {
    const int v = v0 + j * step;
    x0[j] = y0[j] = 0.f;
    if (v < nq + nk && lane < half) {
      const float* src = source(v);
      x0[j] = src[lane * pa];
      y0[j] = src[lane * pa + pb];
    }
  }
  float* cs = sm;
  float* sn = sm + half;
  for (int i = tid; i < half; i += 256) rotary_sincos(a.freq[i], pos, sn[i], cs[i]);
  CT* crow = reinterpret_cast<CT*>(a.cache) + cache_row(a, a.slot[t], pos);
  __syncthreads();
#pragma unroll
  for (int j = 0; j < NPW; ++j) {
    const int v = v0 + j * step;
    if (v >= total) break;
    const float* src = source(v);
    if (v >= nq + nk) {
      CT* dst = crow + nk * a.dp + (v - nq - nk) * a.vp;
      float* vf = a.v_mix ? a.v_first + ((size_t)t * a.G + v - nq - nk) * a.V : nullptr;
      for (int i0 = lane; i0 < a.vp; i0 += 128) {
        float x[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) x[k] = i0 + k * 32 < a.V ? src[i0 + k * 32] : 0.f;
        if (a.v_mix) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (i0 + k * 32 < a.V) {
              if (a.v_mix == 1) vf[i0 + k * 32] = x[k];
              else x[k] = (1.f - a.mix) * x[k] + a.mix * vf[i0 + k * 32];
            }
        }
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (i0 + k * 32 < a.vp) dst[i0 + k * 32] = (CT)x[k];
      }
      continue;
    }
    const bool is_q = v < nq;
    CT* krow = is_q ? nullptr : crow + (v - nq) * a.dp;
    float* qx = is_q && a.qx ? a.qx + ((size_t)t * nq + v) * a.D : nullptr;
    bf16* qf = is_q && a.qf ? (bf16*)a.qf + ((size_t)t * nq + v) * a.q_ld : nullptr;
    const float* nw = is_q ? a.q_norm : a.k_norm;
    float rn = 1.f;
    if (nw) {
      float ss = 0.f;
      for (int i = lane; i < a.D; i += 32) ss = fmaf(src[i], src[i], ss);
      rn = 1.f / sqrtf(warp_sum(ss) / (float)a.D + a.eps);
    }
    auto normed = [&](int i, float x) { return nw ? x * rn * nw[i] : x; };
    auto put = [&](int i, float x) {
      if (krow) krow[i] = (CT)x;
      if (qx) qx[i] = x;
      if (qf) qf[i] = __float2bfloat16(x);
    };
    for (int i = lane; i < half; i += 32) {
      const int e = i * pa, o = e + pb;
      float x = normed(e, i == lane ? x0[j] : src[e]), y = normed(o, i == lane ? y0[j] : src[o]);
      rotate_pair(x, y, sn[i], cs[i]);
      put(e, x);
      put(o, y);
    }
    for (int i = a.R + lane; i < a.D; i += 32) put(i, normed(i, src[i]));
    if (krow)
      for (int i = a.D + lane; i < a.dp; i += 32) krow[i] = (CT)0.f;
    if (qf)
      for (int i = a.D + lane; i < a.q_ld; i += 32) qf[i] = __float2bfloat16(0.f);
  }
  if (a.row > nk * a.dp + a.G * a.vp && blockIdx.y == 0)
    for (int i = nk * a.dp + a.G * a.vp + tid; i < a.row; i += 256) crow[i] = (CT)0.f;
}

// One block: one row, up to QB query vectors of one key head (a head's maps are neighbours), one split of its visible
// positions. Warp w owns vector w's scores (lane = cached row of the tile); for the weighted sums a thread owns one pair of
// value columns for all vectors and every (8 / cw)-th row of the tile, cw = warps that span the columns.
template <typename CT>
__global__ void __launch_bounds__(32 * QB) paged_rows_kernel(const Attn a, const int* rows, int subs, int kld, int vld, int cw) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smraw[];
  constexpr int VE = 16 / sizeof(CT);
  float* qs = reinterpret_cast<float*>(smraw);                    // [QB][dp]
  CT* ks = reinterpret_cast<CT*>(qs + QB * a.dp);                 // [TK][kld]
  CT* vs = ks + TK * kld;                                         // [TK][vld]
  float* ps = reinterpret_cast<float*>(vs + TK * vld);            // [TK][QB]
  float* al = ps + TK * QB;                                       // [QB]
  float* red = al + QB;                                           // [8 / cw - 1][QB][vp] (last reduction)
  const int li = blockIdx.x, g = blockIdx.y / subs, sub = blockIdx.y % subs, sp = blockIdx.z, tid = threadIdx.x;
  const int warp = tid >> 5, lane = tid & 31;
  const int t = rows[li], pos = a.pos[t], slot = a.slot[t];
  const int first = first_visible(a, pos), n = pos + 1 - first;
  const int per = ((n + a.nsplit - 1) / a.nsplit + TK - 1) / TK * TK;
  const int s0 = first + sp * per, s1 = min(pos + 1, s0 + per);
  const int nq = a.H * a.maps, group = nq / a.G;                  // query vectors of a key head
  const int q0 = sub * QB, nv = min(QB, group - q0), qbase = g * group + q0;
  for (int i = tid; i < QB * a.dp; i += 32 * QB) {
    const int q = i / a.dp, d = i - q * a.dp;
    qs[i] = q < nv && d < a.D ? a.qx[((size_t)t * nq + qbase + q) * a.D + d] : 0.f;
  }
  const int krow = a.maps * a.dp, kvec = krow / VE, vvec = a.vp / VE;
  const int kbase = g * krow, vbase = a.G * krow + g * a.vp;
  const int key_map = (q0 + warp) % a.maps;
  const int ncol = a.vp / 2, col = (warp % cw) * 32 + lane, slice = warp / cw, slices = QB / cw;
  float m = -INFINITY, l = 0.f;
  float acc[QB][2];
#pragma unroll
  for (int q = 0; q < QB; ++q) acc[q][0] = acc[q][1] = 0.f;
  for (int k0 = s0; k0 < s1; k0 += TK) {
    const int nk = min(TK, s1 - k0);
    __syncthreads();
    // four rows per warp; their addresses first, so that their loads are in flight together
    constexpr int RW = TK / QB;
    const CT* src[RW];
#pragma unroll
    for (int j = 0; j < RW; ++j) src[j] = reinterpret_cast<const CT*>(a.cache) + cache_row(a, slot, k0 + min(warp + j * QB, nk - 1));
    for (int v = lane; v < kvec + vvec; v += 32) {
      const bool key = v < kvec;
      const int from = key ? kbase + v * VE : vbase + (v - kvec) * VE;
      uint4 x[RW];
#pragma unroll
      for (int j = 0; j < RW; ++j) x[j] = *reinterpret_cast<const uint4*>(src[j] + from);
#pragma unroll
      for (int j = 0; j < RW; ++j) {
        const int r = warp + j * QB;
        *reinterpret_cast<uint4*>(key ? ks + r * kld + v * VE : vs + r * vld + (v - kvec) * VE) = x[j];
      }
    }
    __syncthreads();
    float s4[4] = {0.f, 0.f, 0.f, 0.f};
    if (warp < nv) {
      const CT* kr = ks + lane * kld + key_map * a.dp;
      const float* q = qs + warp * a.dp;
#pragma unroll 4
      for (int v = 0; v < a.dp; v += VE) {
        const uint4 raw = *reinterpret_cast<const uint4*>(kr + v);
        const CT* ke = reinterpret_cast<const CT*>(&raw);
#pragma unroll
        for (int e = 0; e < VE; ++e) s4[e & 3] = fmaf(to_f<CT>(ke[e]), q[v + e], s4[e & 3]);
      }
    }
    float s = ((s4[0] + s4[1]) + (s4[2] + s4[3])) * a.scale;
    if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
    if (lane >= nk) s = -INFINITY;
    const float mn = fmaxf(m, warp_max(s));
    const float alpha = m == -INFINITY ? 0.f : expf(m - mn);
    const float e = lane < nk ? expf(s - mn) : 0.f;
    l = l * alpha + warp_sum(e);
    m = mn;
    ps[lane * QB + warp] = e;
    if (lane == 0) al[warp] = alpha;
    __syncthreads();
#pragma unroll
    for (int q = 0; q < QB; ++q) {
      const float f = al[q];
      acc[q][0] *= f;
      acc[q][1] *= f;
    }
    if (col < ncol)
      for (int r = slice; r < nk; r += slices) {
        const float4 p0 = *reinterpret_cast<const float4*>(ps + r * QB), p1 = *reinterpret_cast<const float4*>(ps + r * QB + 4);
        const float pv[QB] = {p0.x, p0.y, p0.z, p0.w, p1.x, p1.y, p1.z, p1.w};
        const float x0 = to_f<CT>(vs[r * vld + 2 * col]), x1 = to_f<CT>(vs[r * vld + 2 * col + 1]);
#pragma unroll
        for (int q = 0; q < QB; ++q) {
          acc[q][0] = fmaf(pv[q], x0, acc[q][0]);
          acc[q][1] = fmaf(pv[q], x1, acc[q][1]);
        }
      }
  }
  if (slices > 1) {
    if (slice > 0 && col < ncol) {
#pragma unroll
      for (int q = 0; q < QB; ++q) *reinterpret_cast<float2*>(red + ((size_t)(slice - 1) * QB + q) * a.vp + 2 * col) = make_float2(acc[q][0], acc[q][1]);
    }
    __syncthreads();
    if (slice == 0 && col < ncol)
      for (int s = 0; s < slices - 1; ++s)
#pragma unroll
        for (int q = 0; q < QB; ++q) {
          const float2 x = *reinterpret_cast<const float2*>(red + ((size_t)s * QB + q) * a.vp + 2 * col);
          acc[q][0] += x.x;
          acc[q][1] += x.y;
        }
  }
  const size_t base = ((size_t)li * a.nsplit + sp) * nq + qbase;
  if (lane == 0 && warp < nv) {
    a.part_ml[(base + warp) * 2] = m;
    a.part_ml[(base + warp) * 2 + 1] = l;
  }
  if (slice == 0 && col < ncol) {
#pragma unroll
    for (int q = 0; q < QB; ++q)
      if (q < nv) {
        if (2 * col < a.V) a.part_o[(base + q) * a.V + 2 * col] = acc[q][0];
        if (2 * col + 1 < a.V) a.part_o[(base + q) * a.V + 2 * col + 1] = acc[q][1];
      }
  }
}

// Block (listed row, head). rows null: row r itself.
template <typename OutT>
__global__ void __launch_bounds__(128) paged_merge_kernel(const Attn a, const int* rows) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float ws[];       // [maps][nsplit]
  __shared__ float scratch[33];
  constexpr int KEEP = 4;
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nq = a.H * a.maps, ns = a.nsplit;
  if (warp < a.maps) {
    float* w = ws + warp * ns;
    if (a.part_ml) {
      const float* ml = a.part_ml + ((size_t)r * ns * nq + h * a.maps + warp) * 2;
      const float sink = a.sink ? a.sink[h * a.maps + warp] : -INFINITY;
      float mx = sink;
      for (int s = lane; s < ns; s += 32) mx = fmaxf(mx, ml[(size_t)s * nq * 2]);
      mx = warp_max(mx);
      float den = 0.f;
      for (int s = lane; s < ns; s += 32) {
        const float m = ml[(size_t)s * nq * 2];
        const float e = m == -INFINITY ? 0.f : expf(m - mx);
        w[s] = e;
        den += e * ml[(size_t)s * nq * 2 + 1];
      }
      den = warp_sum(den);
      if (a.sink) den += expf(sink - mx);
      __syncwarp();
      for (int s = lane; s < ns; s += 32) w[s] /= den;
    } else if (lane == 0) {
      w[0] = 1.f;
    }
  }
  __syncthreads();
  float o[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = tid + i * 128;
    o[i] = 0.f;
    if (v < a.V) {
      const float* p = a.part_o + ((size_t)r * ns * nq + h * a.maps) * a.V + v;
      float x = 0.f, y = 0.f;
      // an empty split holds zeros: every term is finite
#pragma unroll 8
      for (int s = 0; s < ns; ++s) x = fmaf(ws[s], p[(size_t)s * nq * a.V], x);
      if (a.maps == 2) {
#pragma unroll 8
        for (int s = 0; s < ns; ++s) y = fmaf(ws[ns + s], p[((size_t)s * nq + 1) * a.V], y);
      }
      o[i] = a.maps == 2 ? x - a.lambda * y : x;
      ss = fmaf(o[i], o[i], ss);
    }
  }
  const int t = rows ? rows[r] : r;
  float f = a.head_norm ? a.post / sqrtf(block_sum(ss, scratch) / (float)a.V + a.eps) : a.post;
  if (a.gate >= 0) f /= 1.f + expf(-a.proj[(size_t)t * a.ld + a.gate + h]);
  OutT* dst = reinterpret_cast<OutT*>(a.out) + (size_t)t * a.ldo;
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if (tid + i * 128 < a.V) dst[h * a.V + tid + i * 128] = (OutT)(o[i] * f);
  if (h == a.H - 1)
    for (int v = a.H * a.V + tid; v < a.width; v += 128) dst[v] = (OutT)0.f;
}

bool shape_ok(const Attn* a) {
  return a != nullptr && a->H >= 1 && a->G >= 1 && a->H % a->G == 0 && (a->maps == 1 || a->maps == 2) && a->D >= 1 && a->V >= 1 && a->V <= 512 && a->R >= 0 &&
         (a->R & 1) == 0 && a->R <= a->D && a->dp >= a->D && (a->dp & 7) == 0 && a->vp >= a->V && (a->vp & 7) == 0 && (a->row & 7) == 0 &&
         a->row >= a->G * (a->maps * a->dp + a->vp) && a->cache != nullptr && a->table != nullptr && a->pos != nullptr && a->slot != nullptr &&
         ((uintptr_t)a->cache & 15) == 0 && (a->v_mix == 0 || ((a->v_mix == 1 || a->v_mix == 2) && a->v_first != nullptr));
}

template <typename CT>
int launch_rows(const Attn& a, const int* rows, int nrows, cudaStream_t stream) {
  constexpr int VE = 16 / sizeof(CT);
  const int group = a.H * a.maps / a.G, subs = (group + QB - 1) / QB;
  // padded tile rows: an odd number of 16-byte units, so that the lanes' rows start in different banks
  const int kld = (a.maps * a.dp / VE | 1) * VE, vld = (a.vp / VE | 1) * VE;
  int cw = 1;
  while (cw * 64 < a.vp) cw *= 2;
  const size_t smem = (size_t)QB * a.dp * 4 + (size_t)TK * (kld + vld) * sizeof(CT) + (size_t)(TK * QB + QB) * 4 + (size_t)(QB / cw - 1) * QB * a.vp * 4;
  if (smem > 227 * 1024 || cw > QB || subs * a.G > 65535) return PK_ERR_UNSUPPORTED;
  static PkDeviceOnce once;
  if (PkDeviceOnceGuard g{once}; g.needed()) {
    if (cudaFuncSetAttribute(paged_rows_kernel<CT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    g.done();
  }
  PK_LAUNCH_PDL(paged_rows_kernel<CT>, dim3(nrows, subs * a.G, a.nsplit), dim3(32 * QB), smem, stream, a, rows, subs, kld, vld, cw);
  return PK_OK;
}

}  // namespace

// Rotation, cache append and queries of M rows.
PK_API int pk_paged_prep(const PkPagedAttention* a, int M, cudaStream_t stream) {
  if (!shape_ok(a) || M < 1 || a->proj == nullptr || (a->R > 0 && a->freq == nullptr) || (a->qf != nullptr && a->q_ld < a->D)) return PK_ERR_BAD_ARG;
  const int total = a->H * a->maps + a->G * a->maps + a->G;
  const size_t smem = (size_t)(a->R + 2) * sizeof(float);
  if (smem > 48 * 1024) return PK_ERR_UNSUPPORTED;
  const dim3 few(M, (total + 7) / 8), many(M, (total + 31) / 32), block(256);
  if (M <= 64) {
    if (a->f32) PK_LAUNCH_PDL((paged_prep_kernel<float, 1>), few, block, smem, stream, *a);
    else PK_LAUNCH_PDL((paged_prep_kernel<pk::bf16, 1>), few, block, smem, stream, *a);
  } else {
    if (a->f32) PK_LAUNCH_PDL((paged_prep_kernel<float, 4>), many, block, smem, stream, *a);
    else PK_LAUNCH_PDL((paged_prep_kernel<pk::bf16, 4>), many, block, smem, stream, *a);
  }
  return PK_OK;
}

// Partial attention of the listed rows over nsplit shares of their visible positions, from qx and the cache.
PK_API int pk_paged_rows(const PkPagedAttention* a, const int* rows, int nrows, cudaStream_t stream) {
  if (!shape_ok(a) || rows == nullptr || nrows < 1 || a->qx == nullptr || a->part_o == nullptr || a->part_ml == nullptr || a->nsplit < 1 || a->nsplit > 1024)
    return PK_ERR_BAD_ARG;
  return a->f32 ? launch_rows<float>(*a, rows, nrows, stream) : launch_rows<pk::bf16>(*a, rows, nrows, stream);
}

// Finished outputs of the listed rows (rows null: rows 0 .. nrows - 1).
PK_API int pk_paged_merge(const PkPagedAttention* a, const int* rows, int nrows, cudaStream_t stream) {
  if (!shape_ok(a) || nrows < 1 || a->part_o == nullptr || a->out == nullptr || a->width < a->H * a->V || a->ldo < a->width || (a->gate >= 0 && a->proj == nullptr) || a->nsplit < 1 || a->nsplit > 1024 ||
      (a->part_ml == nullptr && a->nsplit != 1) || a->H > 65535)
    return PK_ERR_BAD_ARG;
  const size_t smem = (size_t)a->maps * a->nsplit * sizeof(float);
  const dim3 grid(nrows, a->H);
  if (a->f32) PK_LAUNCH_PDL(paged_merge_kernel<float>, grid, dim3(128), smem, stream, *a, rows);
  else PK_LAUNCH_PDL(paged_merge_kernel<pk::bf16>, grid, dim3(128), smem, stream, *a, rows);
  return PK_OK;
}
