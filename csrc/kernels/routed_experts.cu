// Routed experts: every token takes the `top` experts with the largest router scores (an optional bias is part of the logits, an
// optional correction per expert counts for the choice alone); an expert is W_down act(W_up x) with act = max(., 0)^2, or W_down (silu(W_gate x) * (W_up x)), and the
// routing weight multiplies either its input (as a factor on the products, which is the same) or its output (as a factor
// behind the activation). The last of the experts may be identities: they have no weights and return their input; what they
// add up to, one factor per token, is left to the norm that follows (sandwich_norm.cu).
//
//   few rows   up: one block row per route, which selects its expert from the router logits itself; down: every output
//              column sums the token's experts, so nothing is scattered or added twice
//   many rows  select, group by expert (segments), gather of the token rows; the two products are grouped tensor-core GEMMs
//              (gemm_bf16.cu) and the sum of a token's rows is part of the next norm (sandwich_norm.cu)
// Scores and weights are fp32.
#include "../common/pk_common.cuh"

namespace {

using namespace pk;

enum { SCORE_SIGMOID = 0, SCORE_SOFTMAX = 1 };
constexpr int kMaxExperts = 512, kMaxTop = 32, WARPS = 8;

struct Router {
  const float* z;      // [tokens, ldz] logits
  int ldz, E, top, score, renorm;      // E: experts and identities
  float scale;
  const float* correction;             // [E] added to the scores for the choice (null: none)
  int real;                            // the first `real` experts have weights
  const float* bias;                   // [E] added to the logits (null: none)
};

// One warp, up to 32 PER experts. Lane j < top gets the j-th best expert and its weight (ties: the lower index first).
template <int PER>
__device__ __forceinline__ void select_experts(const Router& r, int token, int lane, int& expert, float& weight) {
  const float* z = r.z + (size_t)token * r.ldz;
  float v[PER];
#pragma unroll
  for (int i = 0; i < PER; ++i) {
    const int e = i * 32 + lane;
    v[i] = -INFINITY;
    if (i * 32 < r.E && e < r.E) v[i] = fmaxf(z[e] + (r.bias ? r.bias[e] : 0.f), -3.0e38f);
  }
  float zmax = 0.f, den = 1.f, sc[PER];      // v: what the choice compares; sc: scores (kept apart when they differ)
  if (r.score == SCORE_SOFTMAX) {
    zmax = -INFINITY;
    den = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) zmax = fmaxf(zmax, v[i]);
    zmax = warp_max(zmax);
#pragma unroll
    for (int i = 0; i < PER; ++i) den += expf(v[i] - zmax);
    den = warp_sum(den);
  }
  auto score = [&](float x) { return r.score == SCORE_SOFTMAX ? expf(x - zmax) / den : 1.f / (1.f + expf(-x)); };
  if (r.correction) {
#pragma unroll
    for (int i = 0; i < PER; ++i) {
      const int e = i * 32 + lane;
      sc[i] = 0.f;
      if (i * 32 < r.E && e < r.E) {
        sc[i] = score(v[i]);
        v[i] = fmaxf(sc[i] + r.correction[e], -3.0e38f);
      }
    }
  }
  expert = 0;
  weight = 0.f;
  float sum = 0.f;
  for (int j = 0; j < r.top; ++j) {
    float bv = -INFINITY;
    int bi = kMaxExperts;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (v[i] > bv) {
        bv = v[i];
        bi = i * 32 + lane;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) {
        bv = ov;
        bi = oi;
      }
    }
    float own = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i)
      if (i * 32 + lane == bi) {
        v[i] = -INFINITY;
        if (r.correction) own = sc[i];
      }
    const float s = r.correction ? __shfl_sync(0xffffffffu, own, bi & 31) : score(bv);
    sum += s;
    if (lane == j) {
      expert = min(bi, r.E - 1);
      weight = s;
    }
  }
  weight *= r.renorm ? r.scale / (sum + 1e-20f) : r.scale;
}

// Sum of the weights of a token's identities (lane j holds route j).
__device__ __forceinline__ float identity_weight(const Router& r, int lane, int expert, float weight) {
  return warp_sum(lane < r.top && expert >= r.real ? weight : 0.f);
}

template <typename T>
struct Vec;      // 16 bytes of a row
template <>
struct Vec<bf16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void get(const uint4& u, float (&f)[8]) {
    const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
};
template <>
struct Vec<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void get(const uint4& u, float (&f)[4]) {
    f[0] = __uint_as_float(u.x);
    f[1] = __uint_as_float(u.y);
    f[2] = __uint_as_float(u.z);
    f[3] = __uint_as_float(u.w);
  }
};

// acc0 / acc1 += two weight rows . x over this warp's slice of K; U 16-byte pieces of each row in flight (few registers and
// many warps stream faster than the reverse).
template <typename T, int U>
__device__ __forceinline__ void dot_rows(const T* w0, const T* w1, const T* x, int K, int slice, int slices, int lane, float& acc0, float& acc1) {
  constexpr int VN = Vec<T>::N;
  const int stride = 32 * VN * slices;
  int k = (slice * 32 + lane) * VN;
  uint4 a[U], b[U];
#pragma unroll
  for (int u = 0; u < U; ++u) {
    a[u] = b[u] = make_uint4(0, 0, 0, 0);
    if (k + u * stride < K) {
      a[u] = ld_stream_u4(w0 + k + u * stride);
      b[u] = ld_stream_u4(w1 + k + u * stride);
    }
  }
  while (k < K) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int kk = k + u * stride;
      if (kk < K) {
        float fa[VN], fb[VN], fx[VN];
        Vec<T>::get(a[u], fa);
        Vec<T>::get(b[u], fb);
        if (kk + U * stride < K) {
          a[u] = ld_stream_u4(w0 + kk + U * stride);
          b[u] = ld_stream_u4(w1 + kk + U * stride);
        }
        Vec<T>::get(*reinterpret_cast<const uint4*>(x + kk), fx);
#pragma unroll
        for (int e = 0; e < VN; ++e) {
          acc0 = fmaf(fa[e], fx[e], acc0);
          acc1 = fmaf(fb[e], fx[e], acc1);
        }
      }
    }
    k += U * stride;
  }
}

// Sum of the slices of a row pair in lane 0 of its first warp.
__device__ __forceinline__ void join_slices(float (*part)[2], int warp, int lane, int slice, int slices, float& a0, float& a1) {
  a0 = warp_sum(a0);
  a1 = warp_sum(a1);
  if (slices > 1) {
    if (lane == 0) {
      part[warp][0] = a0;
      part[warp][1] = a1;
    }
    __syncthreads();
    if (slice == 0)
      for (int s = 1; s < slices; ++s) {
        a0 += part[warp + s][0];
        a1 += part[warp + s][1];
      }
  }
}

struct RowsParams {
  Router r;
  const void* x;        // [tokens, ldx]
  int ldx;
  const void* w;        // up: [real, N, K], gated: [real, N gate rows and N up rows, K]; down: [real, w_rows, K]
  int N, K, w_rows, slices, scale_after, gated;
  int* ids;             // [tokens, top] chosen experts: written by up, read by down
  float* skip_w;        // [tokens] weight of the identities (null: there are none)
  void* y;              // up: [tokens * top, ldy] hidden; down: [tokens, ldy] fp32
  int ldy;
};

template <typename T, int PER>
__global__ void __launch_bounds__(32 * WARPS) expert_up_rows_kernel(const RowsParams p) {
  __shared__ float part[WARPS][2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_trigger();
  pdl_wait();
  const int route = blockIdx.x, t = route / p.r.top, j = route - t * p.r.top;
  int e;
  float s;
  select_experts<PER>(p.r, t, lane, e, s);
  if (p.skip_w && blockIdx.y == 0 && j == 0 && warp == 0) {
    const float f = identity_weight(p.r, lane, e, s);
    if (lane == 0) p.skip_w[t] = f;
  }
  e = __shfl_sync(0xffffffffu, e, j);
  s = __shfl_sync(0xffffffffu, s, j);
  if (blockIdx.y == 0 && threadIdx.x == 0) p.ids[route] = e;
  if (e >= p.r.real) return;
  const int g = blockIdx.y * (WARPS / p.slices) + warp / p.slices, slice = warp % p.slices;
  const int n0 = p.gated ? g : 2 * g, n1 = p.gated ? p.N + g : min(2 * g + 1, p.N - 1);
  const bool live = n0 < p.N;
  float a0 = 0.f, a1 = 0.f;
  if (live) {
    const T* w = (const T*)p.w + (size_t)e * p.w_rows * p.K;
    dot_rows<T, 2>(w + (size_t)n0 * p.K, w + (size_t)n1 * p.K, (const T*)p.x + (size_t)t * p.ldx, p.K, slice, p.slices, lane, a0, a1);
  }
  join_slices(part, warp, lane, slice, p.slices, a0, a1);
  if (live && slice == 0 && lane == 0) {
    const float s0 = p.scale_after ? 1.f : s, s1 = p.scale_after ? s : 1.f;
    T* y = (T*)p.y + (size_t)route * p.ldy;
    if (p.gated) {
      a0 *= s0;
      y[n0] = (T)(a0 / (1.f + expf(-a0)) * (a1 * s0) * s1);
      return;
    }
    a0 = fmaxf(a0 * s0, 0.f);
    a1 = fmaxf(a1 * s0, 0.f);
    y[n0] = (T)(a0 * a0 * s1);
    if (2 * g + 1 < p.N) y[n1] = (T)(a1 * a1 * s1);
  }
}

template <typename T>
__global__ void __launch_bounds__(32 * WARPS) expert_down_rows_kernel(const RowsParams p) {
  __shared__ float part[WARPS][2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int g = blockIdx.y * (WARPS / p.slices) + warp / p.slices, slice = warp % p.slices;
  const int n0 = 2 * g, n1 = min(2 * g + 1, p.N - 1);
  const bool live = n0 < p.N;
  float a0 = 0.f, a1 = 0.f;
  if (live)
    for (int j = 0; j < p.r.top; ++j) {
      const int route = t * p.r.top + j, e = p.ids[route];
      if (e >= p.r.real) continue;
      const T* w = (const T*)p.w + (size_t)e * p.w_rows * p.K;
      dot_rows<T, 2>(w + (size_t)n0 * p.K, w + (size_t)n1 * p.K, (const T*)p.x + (size_t)route * p.ldx, p.K, slice, p.slices, lane, a0, a1);
    }
  join_slices(part, warp, lane, slice, p.slices, a0, a1);
  if (live && slice == 0 && lane == 0) {
    float* y = (float*)p.y + (size_t)t * p.ldy;
    y[n0] = a0;
    if (2 * g + 1 < p.N) y[n1] = a1;
  }
}

// One warp per token.
__global__ void __launch_bounds__(128) select_kernel(const Router r, int T, int* ids, float* weights, float* skip_w) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  int e;
  float w;
  select_experts<kMaxExperts / 32>(r, t, lane, e, w);
  if (lane < r.top) {
    ids[(size_t)t * r.top + lane] = e;
    weights[(size_t)t * r.top + lane] = w;
  }
  if (skip_w) {
    const float f = identity_weight(r, lane, e, w);
    if (lane == 0) skip_w[t] = f;
  }
}

// One block: segment of every expert, place of every route in expert order (the order inside a segment is arbitrary: rows
// of a product do not depend on their neighbours; -1 for identities), and the routing weight in that order.
__global__ void __launch_bounds__(1024) group_kernel(const int* ids, const float* weights, int R, int E, int real, int* seg, int* place, float* row_scale) {
  pdl_trigger();
  pdl_wait();
  __shared__ int cnt[kMaxExperts], warp_tot[32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  if (tid < kMaxExperts) cnt[tid] = 0;
  __syncthreads();
  for (int r = tid; r < R; r += 1024) atomicAdd(&cnt[ids[r]], 1);
  __syncthreads();
  const int own = tid < E ? cnt[tid] : 0;
  int run = own;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int v = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += v;
  }
  if (lane == 31) warp_tot[warp] = run;
  __syncthreads();
  for (int w = 0; w < warp; ++w) run += warp_tot[w];
  __syncthreads();
  if (tid < E) {
    cnt[tid] = run - own;
    if (tid < real) seg[tid] = run - own;
    if (tid == real - 1) seg[real] = run;
  }
  __syncthreads();
  for (int r = tid; r < R; r += 1024) {
    if (ids[r] >= real) {
      place[r] = -1;
      continue;
    }
    const int at = atomicAdd(&cnt[ids[r]], 1);
    place[r] = at;
    row_scale[at] = weights[r];
  }
}

// Token rows in expert order: out[place[t * top + j]] = x[t]. One block per token.
__global__ void __launch_bounds__(128) gather_kernel(const bf16* x, int ldx, int K, int top, const int* place, bf16* out) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const uint4* src = reinterpret_cast<const uint4*>(x + (size_t)t * ldx);
  for (int v = threadIdx.x; v < K / 8; v += 128) {
    const uint4 u = src[v];
    for (int j = 0; j < top; ++j) {
      const int at = place[(size_t)t * top + j];
      if (at >= 0) reinterpret_cast<uint4*>(out + (size_t)at * K)[v] = u;
    }
  }
}

bool router_ok(const Router& r) {
  return r.z != nullptr && r.E >= 1 && r.E <= kMaxExperts && r.top >= 1 && r.top <= kMaxTop && r.top <= r.E && r.ldz >= r.E && r.real >= 1 && r.real <= r.E &&
         (r.score == SCORE_SIGMOID || r.score == SCORE_SOFTMAX);
}

int pick_slices(long long pairs, int K, int vec, int sm_count) {
  const long long want = (long long)(sm_count > 0 ? sm_count : 148) * 32;
  int s = 1;
  while (s < WARPS && pairs * s < want && K >= 64 * vec * s * 2) s *= 2;
  return s;
}

}  // namespace

// Hidden rows of T tokens' experts. logits [T, ldz]; x [T, ldx] and w_up [E - identity, N, K] (gated: N gate rows, then N up
// rows each) bf16, or fp32 when `f32`; hidden [T * top, ldh] of the same type; ids [T, top] out. K a multiple of 8, rows
// 16-byte aligned. score 0 sigmoid, 1 softmax; correction, bias [E] or null; renorm: the chosen weights are divided by their sum;
// scale: factor on them; scale_after: weight on the output instead of the input; identity: how many of the E experts are
// identities (skip_w [T] out, the sum of their weights).
PK_API int pk_expert_up_rows(const float* logits, int ldz, int E, int top, int score, int renorm, float scale, const float* correction, const float* bias, int identity,
                             float* skip_w, int scale_after, int gated, const void* x, int ldx, int T, const void* w_up, int N, int K, int f32,
                             int* ids, void* hidden, int ldh, int sm_count, cudaStream_t stream) {
  Router r{logits, ldz, E, top, score, renorm, scale, correction, E - identity, bias};
  if (!router_ok(r) || T < 1 || N < 1 || K < 8 || (K & 7) != 0 || ldx < K || (ldx & 7) != 0 || ldh < N || x == nullptr || w_up == nullptr || ids == nullptr ||
      hidden == nullptr || ((uintptr_t)x & 15) != 0 || ((uintptr_t)w_up & 15) != 0 || identity < 0 || (identity > 0 && skip_w == nullptr))
    return PK_ERR_BAD_ARG;
  RowsParams p{r, x, ldx, w_up, N, K, gated ? 2 * N : N, 1, scale_after, gated, ids, skip_w, hidden, ldh};
  const int pairs = gated ? N : (N + 1) / 2;
  p.slices = pick_slices((long long)pairs * T * top, K, f32 ? 4 : 8, sm_count);
  const dim3 grid(T * top, (pairs + WARPS / p.slices - 1) / (WARPS / p.slices));
  if (grid.y > 65535) return PK_ERR_UNSUPPORTED;
  const dim3 block(32 * WARPS);
  if (f32) PK_LAUNCH_PDL((expert_up_rows_kernel<float, kMaxExperts / 32>), grid, block, (size_t)0, stream, p);
  else if (E <= 64) PK_LAUNCH_PDL((expert_up_rows_kernel<pk::bf16, 2>), grid, block, (size_t)0, stream, p);
  else PK_LAUNCH_PDL((expert_up_rows_kernel<pk::bf16, kMaxExperts / 32>), grid, block, (size_t)0, stream, p);
  return PK_OK;
}

// y [T, ldy] fp32 = sum over the token's experts of W_down hidden; w_down [real, w_rows, K] (the first N rows of each are
// used; ids from `real` on add nothing).
PK_API int pk_expert_down_rows(const int* ids, int top, int real, const void* hidden, int ldh, int T, const void* w_down, int N, int w_rows, int K, int f32,
                               float* y, int ldy, int sm_count, cudaStream_t stream) {
  if (ids == nullptr || top < 1 || top > kMaxTop || T < 1 || N < 1 || w_rows < N || K < 8 || (K & 7) != 0 || ldh < K || (ldh & 7) != 0 || ldy < N ||
      hidden == nullptr || w_down == nullptr || y == nullptr || ((uintptr_t)hidden & 15) != 0 || ((uintptr_t)w_down & 15) != 0)
    return PK_ERR_BAD_ARG;
  RowsParams p{Router{nullptr, 0, 0, top, 0, 0, 0.f, nullptr, real, nullptr}, hidden, ldh, w_down, N, K, w_rows, 1, 0, 0, (int*)ids, nullptr, y, ldy};
  const int pairs = (N + 1) / 2;
  p.slices = pick_slices((long long)pairs * T, K, f32 ? 4 : 8, sm_count);
  const dim3 grid(T, (pairs + WARPS / p.slices - 1) / (WARPS / p.slices));
  if (grid.y > 65535) return PK_ERR_UNSUPPORTED;
  if (f32) PK_LAUNCH_PDL(expert_down_rows_kernel<float>, grid, dim3(32 * WARPS), (size_t)0, stream, p);
  else PK_LAUNCH_PDL(expert_down_rows_kernel<pk::bf16>, grid, dim3(32 * WARPS), (size_t)0, stream, p);
  return PK_OK;
}

// Routes of T tokens grouped by expert: ids, weights [T, top]; seg [E - identity + 1]; place [T, top]; row_scale [T * top];
// rows [T * top, K] bf16 = the tokens' x in expert order (K a multiple of 8); skip_w as above.
PK_API int pk_expert_group(const float* logits, int ldz, int E, int top, int score, int renorm, float scale, const float* correction, const float* bias, int identity,
                           float* skip_w, int T, int* ids, float* weights, int* seg, int* place, float* row_scale, const void* x, int ldx, int K,
                           void* rows, cudaStream_t stream) {
  Router r{logits, ldz, E, top, score, renorm, scale, correction, E - identity, bias};
  if (!router_ok(r) || T < 1 || identity < 0 || (identity > 0 && skip_w == nullptr) || ids == nullptr || weights == nullptr || seg == nullptr ||
      place == nullptr || row_scale == nullptr || x == nullptr || rows == nullptr || K < 8 || (K & 7) != 0 || (ldx & 7) != 0 || ldx < K || ((uintptr_t)x & 15) != 0 || ((uintptr_t)rows & 15) != 0)
    return PK_ERR_BAD_ARG;
  PK_LAUNCH_PDL(select_kernel, dim3((T + 3) / 4), dim3(128), (size_t)0, stream, r, T, ids, weights, skip_w);
  PK_LAUNCH_PDL(group_kernel, dim3(1), dim3(1024), (size_t)0, stream, (const int*)ids, (const float*)weights, T * top, E, E - identity, seg, place, row_scale);
  PK_LAUNCH_PDL(gather_kernel, dim3(T), dim3(128), (size_t)0, stream, (const pk::bf16*)x, ldx, K, top, (const int*)place, (pk::bf16*)rows);
  return PK_OK;
}
