// Selective scan of Mamba: per channel c and state n
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,     y_c = sum_n S[c, n] C_n + D_c x_c,     out_c = y_c silu(z_c)
// with x behind a short causal convolution per channel and SiLU, dt_c = softplus(W_dt d + bias), and d, B, C from a product with x.
// State [slots, inner, state] fp32; the convolution's last inputs in a ring [slot][position modulo (taps - 1)][channel], as in the
// state space of ssd.cu: a token writes one entry, nothing shifts, inputs before position 0 are zero by position. Nothing is
// cleared on reuse of a slot: a portion that starts at position 0 starts from zero.
//
//   conv   x of all rows, into the type of the model (the operand of the product that yields d, B, C)
//   split  d as the sum of two bf16 terms side by side, so that W_dt d of many rows on the tensor cores keeps 16 bits of d
//   rows   portions of a few tokens: LN lanes per channel with NP states each, W_dt d in the same kernel (fp32 sums)
//   tiles  long portions: the same lanes walk the tokens in tiles of 16 (8); the tile's B and C arrive by cp.async and its dt and x through
//          registers while the tile before is worked on; the sums over a channel's lanes are taken for LN tokens at a time (every
//          exchange halves the number of partial sums); the outputs of a tile are gated and stored together
// Everything but x and W_dt is fp32. A decay close to 1 that is rounded to fp32 is off by the same few 2^-25 at every step of a long
// memory; fp32 models therefore take what a state loses, exp(.) - 1, instead.
#include "../common/pk_vec.cuh"

// Plain data mirrored by the Python bindings.
struct PkSelectiveScan {
  const float* proj;       // [rows, ld]: x at column ox, z at oz
  const void* xc;          // [rows, ldx] x behind its convolution (model's type); conv writes it
  const float* dbc;        // [rows, ldb]: d | B | C
  const float* dt;         // [rows, ldt] W_dt d (tiles)
  const void* w_dt;        // [inner, ldw] (rows): `rank` columns, zeros up to a multiple of 8
  const float* dt_bias;    // [inner]
  const float* A;          // [inner, N], negative; times log2(e) when the model is in bf16
  const float* skip;       // [inner]
  const float* cw;         // [inner, taps], the last tap is the current token's
  const float* cb;         // [inner]
  float* S;                // [slots, inner, N]
  float* ring;             // [slots, taps - 1, inner]
  void* out;               // [rows, ldo], columns from inner on zero
  const int* pos;
  const int* slot;
  int ld, ox, oz, ldx, ldb, ldt, ldw, ldo, inner, N, rank, taps, f32;
};

namespace {

using namespace pk;

constexpr int THREADS = 128;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// max(z, 0) + log1p(e), e = exp(-|z|); log1p(e) = 2 artanh(s) = 2 (s + s^3 / 3 + s^5 / 5 + ...), s = e / (2 + e) <= 1 / 3.
__device__ __forceinline__ float softplus_series(float z) {
  const float e = expf(-fabsf(z)), s = __fdividef(e, 2.f + e), q = s * s;
  float p = 1.f / 15.f;
  p = fmaf(p, q, 1.f / 13.f);
  p = fmaf(p, q, 1.f / 11.f);
  p = fmaf(p, q, 1.f / 9.f);
  p = fmaf(p, q, 1.f / 7.f);
  p = fmaf(p, q, 1.f / 5.f);
  p = fmaf(p, q, 1.f / 3.f);
  p = fmaf(p * q, s, s);
  return fmaxf(z, 0.f) + 2.f * p;
}

// s exp(dt A)
template <typename T>
__device__ __forceinline__ float decayed(float dt, float a, float s) {
  return sizeof(T) == 4 ? fmaf(expm1f(dt * a), s, s) : ex2(dt * a) * s;
}

template <typename T>
__device__ __forceinline__ float silu_of(float z) {      // as exact as the type it enters
  return sizeof(T) == 4 ? z / (1.f + expf(-z)) : __fdividef(z, 1.f + __expf(-z));
}

__device__ __forceinline__ float* ring_at(const PkSelectiveScan& p, int slot, int pos) {
  return p.ring + ((size_t)slot * (p.taps - 1) + pos % (p.taps - 1)) * p.inner;
}

// ---------------------------------------------------------------------------------------
// convolution

// Block: 128 groups of VW channels, `per` consecutive rows; a window of the last TAPS inputs moves along (TAPS 0: any number, every
// input is fetched for every row). Rows of one portion have one slot and follow each other.
template <typename T, int TAPS, int VW>
__global__ void __launch_bounds__(THREADS) conv_kernel(const PkSelectiveScan p, int rows, int per) {
  pdl_trigger();
  const int c = (blockIdx.y * THREADS + threadIdx.x) * VW, r0 = blockIdx.x * per, r1 = min(r0 + per, rows);
  T* out = (T*)const_cast<void*>(p.xc);
  constexpr int NT = TAPS > 0 ? TAPS : 1;
  float w[NT][VW], b[VW];
  if (c < p.inner) {
    load_f32<VW>(p.cb + c, b);
    if (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int k = 0; k < VW; ++k) w[j][k] = p.cw[(size_t)(c + k) * NT + j];
    }
  }
  pdl_wait();
  if (c >= p.ldx) return;
  if (c >= p.inner) {      // padding (a group never straddles: inner is a multiple of VW)
    for (int r = r0; r < r1; ++r)
#pragma unroll
      for (int k = 0; k < VW; ++k)
        if (c + k < p.ldx) out[(size_t)r * p.ldx + c + k] = (T)0.f;
    return;
  }
  auto earlier = [&](int r, int slot, int pos, int lag, float (&v)[VW]) {      // input `lag` >= 1 tokens before row r
#pragma unroll
    for (int k = 0; k < VW; ++k) v[k] = 0.f;
    if (lag > pos) return;
    if (r >= lag && p.slot[r - lag] == slot) load_f32<VW>(p.proj + (size_t)(r - lag) * p.ld + p.ox + c, v);
    else load_f32<VW>(ring_at(p, slot, pos - lag) + c, v);
  };
  float win[NT][VW];
  constexpr int AHEAD = TAPS > 0 ? 4 : 1;      // rows whose loads are in flight together
  int last = -1;
  for (int ra = r0; ra < r1; ra += AHEAD) {
    float x[AHEAD][VW];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) load_f32<VW>(p.proj + (size_t)min(ra + i, r1 - 1) * p.ld + p.ox + c, x[i]);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      const int r = ra + i;
      if (r >= r1) break;
      const int slot = p.slot[r], pos = p.pos[r];
      float y[VW];
#pragma unroll
      for (int k = 0; k < VW; ++k) y[k] = b[k];
      if (TAPS > 0) {
        if (slot != last) {
#pragma unroll
          for (int j = 0; j + 1 < NT; ++j) earlier(r, slot, pos, NT - 1 - j, win[j]);
          last = slot;
        }
#pragma unroll
        for (int k = 0; k < VW; ++k) win[NT - 1][k] = x[i][k];
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
          for (int k = 0; k < VW; ++k) y[k] = fmaf(w[j][k], win[j][k], y[k]);
#pragma unroll
        for (int j = 0; j + 1 < NT; ++j)
#pragma unroll
          for (int k = 0; k < VW; ++k) win[j][k] = win[j + 1][k];
      } else {
        for (int j = 0; j < p.taps; ++j) {
          float v[VW];
          if (j + 1 < p.taps) earlier(r, slot, pos, p.taps - 1 - j, v);
#pragma unroll
          for (int k = 0; k < VW; ++k) y[k] = fmaf(p.cw[(size_t)(c + k) * p.taps + j], j + 1 < p.taps ? v[k] : x[i][k], y[k]);
        }
      }
#pragma unroll
      for (int k = 0; k < VW; ++k) y[k] = silu_of<T>(y[k]);
      store<VW>(out + (size_t)r * p.ldx + c, y);
    }
  }
}

// d [rows, rank] fp32 -> [rows, 2 kp] bf16: leading terms, then remainders, both padded with zeros.
__global__ void __launch_bounds__(256) split_kernel(const float* d, int ldd, int rank, int kp, int rows, bf16* out) {
  pdl_trigger();
  pdl_wait();
  const long long n = (long long)rows * kp;
  for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
    const int r = (int)(i / kp), k = (int)(i - (long long)r * kp);
    const float v = k < rank ? d[(size_t)r * ldd + k] : 0.f;
    const bf16 hi = __float2bfloat16(v);
    out[(size_t)r * 2 * kp + k] = hi;
    out[(size_t)r * 2 * kp + kp + k] = __float2bfloat16(v - __bfloat162float(hi));
  }
}

// ---------------------------------------------------------------------------------------
// recurrence

template <typename T>
__device__ __forceinline__ float to_f(T v) { return (float)v; }
template <>
__device__ __forceinline__ float to_f<bf16>(bf16 v) { return __bfloat162float(v); }

// NP states of a channel from state n0 on.
template <int NP>
__device__ __forceinline__ void load_states(const float* row, int n0, int N, float (&v)[NP]) {
  if (NP % 4 == 0 && (N & 3) == 0) {
#pragma unroll
    for (int k = 0; k < NP; k += 4) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (n0 + k < N) x = *reinterpret_cast<const float4*>(row + n0 + k);
      v[k] = x.x; v[k + 1] = x.y; v[k + 2] = x.z; v[k + 3] = x.w;
    }
  } else {
#pragma unroll
    for (int k = 0; k < NP; ++k) v[k] = n0 + k < N ? row[n0 + k] : 0.f;
  }
}
template <int NP>
__device__ __forceinline__ void store_states(float* row, int n0, int N, const float (&v)[NP]) {
  if (NP % 4 == 0 && (N & 3) == 0) {
#pragma unroll
    for (int k = 0; k < NP; k += 4)
      if (n0 + k < N) *reinterpret_cast<float4*>(row + n0 + k) = make_float4(v[k], v[k + 1], v[k + 2], v[k + 3]);
  } else {
#pragma unroll
    for (int k = 0; k < NP; ++k)
      if (n0 + k < N) row[n0 + k] = v[k];
  }
}

// Block: THREADS / LN channels of one short portion.
template <typename T, int NP, int LN>
__global__ void __launch_bounds__(THREADS) scan_rows_kernel(const PkSelectiveScan p, const int4* seqs) {
  constexpr int CB = THREADS / LN, VE = 16 / sizeof(T), AHEAD = 4;
  extern __shared__ float sm[];
  const int4 sq = seqs[blockIdx.y];            // first row, tokens, slot, first position
  const int tid = threadIdx.x, l = tid % LN, c = blockIdx.x * CB + tid / LN, n0 = l * NP;
  const bool live = c < p.inner;
  const int kw = (p.rank + 7) & ~7;
  float* d = sm;                               // [kw] input of W_dt
  float* B = d + kw;                           // [LN * NP] each
  float* C = B + LN * NP;
  // weights first: no kernel writes them
  const T* wrow = (const T*)p.w_dt + (size_t)(live ? c : 0) * p.ldw;
  uint4 first[AHEAD];
#pragma unroll
  for (int i = 0; i < AHEAD; ++i) {
    const int k = (l + i * LN) * VE;
    first[i] = live && k < kw ? ld_stream_u4(wrow + k) : make_uint4(0, 0, 0, 0);
  }
  float a[NP];
#pragma unroll
  for (int k = 0; k < NP; ++k) a[k] = 0.f;
  if (live) load_states<NP>(p.A + (size_t)c * p.N, n0, p.N, a);
  const float bias = live ? p.dt_bias[c] : 0.f, skip = live ? p.skip[c] : 0.f;
  pdl_trigger();
  pdl_wait();
  float s[NP];
#pragma unroll
  for (int k = 0; k < NP; ++k) s[k] = 0.f;
  float* Sp = p.S + ((size_t)sq.z * p.inner + (live ? c : 0)) * p.N;
  if (live && sq.w > 0) load_states<NP>(Sp, n0, p.N, s);
  for (int t = 0; t < sq.y; ++t) {
    const size_t row = (size_t)sq.x + t;
    const float* src = p.dbc + row * p.ldb;
    for (int i = tid; i < kw; i += THREADS) d[i] = i < p.rank ? src[i] : 0.f;
    for (int i = tid; i < LN * NP; i += THREADS) {
      B[i] = i < p.N ? src[p.rank + i] : 0.f;
      C[i] = i < p.N ? src[p.rank + p.N + i] : 0.f;
    }
    const float x = live ? to_f<T>(((const T*)p.xc)[row * p.ldx + c]) : 0.f;
    float z = 0.f, in = 0.f;
    if (live && l == 0) {
      z = p.proj[row * p.ld + p.oz + c];
      if (sq.y - 1 - t < p.taps - 1) in = p.proj[row * p.ld + p.ox + c];
    }
    __syncthreads();
    float dot = 0.f;
    auto add = [&](const uint4& u, int k) {
      const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
      for (int i = 0; i < VE; ++i) dot = fmaf(to_f<T>(e[i]), d[k + i], dot);
    };
    if (live) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if ((l + i * LN) * VE < kw) add(first[i], (l + i * LN) * VE);
#pragma unroll 4
      for (int k = (l + AHEAD * LN) * VE; k < kw; k += LN * VE) add(*reinterpret_cast<const uint4*>(wrow + k), k);
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
    const float dt = softplus_series(dot + bias), u = dt * x;
    float y = 0.f;
#pragma unroll
    for (int k = 0; k < NP; ++k) {
      s[k] = fmaf(u, B[n0 + k], decayed<T>(dt, a[k], s[k]));
      y = fmaf(s[k], C[n0 + k], y);
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (live && l == 0) {
      T* out = (T*)p.out + row * p.ldo;
      out[c] = (T)(fmaf(skip, x, y) * silu_of<T>(z));
      if (sq.y - 1 - t < p.taps - 1) ring_at(p, sq.z, sq.w + t)[c] = in;
    }
    if (blockIdx.x == gridDim.x - 1)
      for (int i = p.inner + tid; i < p.ldo; i += THREADS) ((T*)p.out)[row * p.ldo + i] = (T)0.f;
    if (t + 1 < sq.y) __syncthreads();
  }
  if (live) store_states<NP>(Sp, n0, p.N, s);
}

// Sums of v[i] over the lanes of a group of G for i < G: lane l of the group gets the sum of v[l].
template <int G>
__device__ __forceinline__ float group_sums(float (&v)[G], int l) {
#pragma unroll
  for (int o = G / 2; o > 0; o >>= 1) {
    const bool up = l & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float give = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

__device__ __forceinline__ void async_f32(float* dst, const float* src, bool in) {      // 4 bytes, or zero
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(a), "l"(src), "r"(in ? 4 : 0) : "memory");
}

// Block: THREADS / LN channels of one long portion, all its tokens.
template <typename T, int NP, int LN>
__global__ void __launch_bounds__(THREADS) scan_tiles_kernel(const PkSelectiveScan p, const int4* seqs) {
  pdl_trigger();
  pdl_wait();
  constexpr int CB = THREADS / LN, NS = LN * NP, TT = NS > 128 ? 8 : 16, G = LN < TT ? LN : TT;      // TT: tokens of a tile
  constexpr int ITEMS = (TT * CB + THREADS - 1) / THREADS;      // (token, channel) pairs of a tile per thread
  __shared__ __align__(16) float Bs[2][TT][NS], Cs[2][TT][NS];
  __shared__ float2 du[TT][CB];                                 // dt, dt x
  __shared__ float ys[TT][CB];
  const int4 sq = seqs[blockIdx.y];
  const int tid = threadIdx.x, l = tid % LN, ch = tid / LN, c0 = blockIdx.x * CB, c = c0 + ch, n0 = l * NP;
  const bool live = c < p.inner;
  const int n = sq.y;
  float a[NP], s[NP];
#pragma unroll
  for (int k = 0; k < NP; ++k) a[k] = s[k] = 0.f;
  float* Sp = p.S + ((size_t)sq.z * p.inner + (live ? c : 0)) * p.N;
  if (live) {
    load_states<NP>(p.A + (size_t)c * p.N, n0, p.N, a);
    if (sq.w > 0) load_states<NP>(Sp, n0, p.N, s);
  }
  // what a thread stages of a tile: dt and x (and z, the raw x for its epilogue) of its pairs
  float dt[ITEMS], x[ITEMS], z[ITEMS], x_now[ITEMS], z_now[ITEMS];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int e = tid + i * THREADS, t = t0 + e / CB, cc = c0 + e % CB;
      dt[i] = x[i] = z[i] = 0.f;
      if (e < TT * CB && t < n && cc < p.inner) {
        const size_t row = (size_t)sq.x + t;
        dt[i] = p.dt[row * p.ldt + cc];
        x[i] = to_f<T>(((const T*)p.xc)[row * p.ldx + cc]);
        z[i] = p.proj[row * p.ld + p.oz + cc];
      }
    }
  };
  auto fetch_bc = [&](int t0, int b) {
    for (int e = tid; e < TT * NS; e += THREADS) {
      const int t = e / NS, k = e % NS;
      const bool in = t0 + t < n && k < p.N;
      const float* src = p.dbc + ((size_t)sq.x + min(t0 + t, n - 1)) * p.ldb + p.rank + min(k, p.N - 1);
      async_f32(&Bs[b][t][k], src, in);
      async_f32(&Cs[b][t][k], src + p.N, in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float bias[ITEMS], skip[ITEMS];
#pragma unroll
  for (int i = 0; i < ITEMS; ++i) {
    const int cc = c0 + (tid + i * THREADS) % CB;
    bias[i] = cc < p.inner ? p.dt_bias[cc] : 0.f;
    skip[i] = cc < p.inner ? p.skip[cc] : 0.f;
  }
  fetch_bc(0, 0);
  fetch(0);
  for (int t0 = 0, b = 0; t0 < n; t0 += TT, b ^= 1) {
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int e = tid + i * THREADS;
      x_now[i] = x[i];
      z_now[i] = z[i];
      if (e < TT * CB) {
        const float d = t0 + e / CB < n ? softplus_series(dt[i] + bias[i]) : 0.f;      // a token behind the end changes nothing
        du[e / CB][e % CB] = make_float2(d, d * x[i]);
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (t0 + TT < n) {
      fetch_bc(t0 + TT, b ^ 1);
      fetch(t0 + TT);
    }
#pragma unroll 1
    for (int tg = 0; tg < TT; tg += G) {
      float y[G];
#pragma unroll
      for (int i = 0; i < G; ++i) {
        const float2 q = du[tg + i][ch];
        float B[NP], C[NP];
        load_states<NP>(Bs[b][tg + i], n0, NS, B);
        load_states<NP>(Cs[b][tg + i], n0, NS, C);
        y[i] = 0.f;
#pragma unroll
        for (int k = 0; k < NP; ++k) {
          s[k] = fmaf(q.y, B[k], decayed<T>(q.x, a[k], s[k]));
          y[i] = fmaf(s[k], C[k], y[i]);
        }
      }
      float sum = group_sums<G>(y, l);
#pragma unroll
      for (int o = G; o < LN; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (l < G) ys[tg + l][ch] = sum;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < ITEMS; ++i) {
      const int e = tid + i * THREADS, t = t0 + e / CB, cc = c0 + e % CB;
      if (e < TT * CB && t < n && cc < p.inner) {
        const size_t row = (size_t)sq.x + t;
        ((T*)p.out)[row * p.ldo + cc] = (T)(fmaf(skip[i], x_now[i], ys[e / CB][e % CB]) * silu_of<T>(z_now[i]));
        if (n - 1 - t < p.taps - 1) ring_at(p, sq.z, sq.w + t)[cc] = p.proj[row * p.ld + p.ox + cc];
      }
    }
    if (blockIdx.x == gridDim.x - 1 && p.ldo > p.inner) {
      const int pad = p.ldo - p.inner;
      for (int e = tid; e < TT * pad; e += THREADS)
        if (t0 + e / pad < n) ((T*)p.out)[((size_t)sq.x + t0 + e / pad) * p.ldo + p.inner + e % pad] = (T)0.f;
    }
  }
  if (live) store_states<NP>(Sp, n0, p.N, s);
}

template <typename T, int NP, int LN>
int launch_scan(const PkSelectiveScan& p, const int4* seqs, int nseq, bool tiles, cudaStream_t stream) {
  constexpr int CB = THREADS / LN;
  const dim3 grid((p.inner + CB - 1) / CB, nseq);
  if (tiles) {
    PK_LAUNCH_PDL((scan_tiles_kernel<T, NP, LN>), grid, dim3(THREADS), (size_t)0, stream, p, seqs);
  } else {
    const size_t smem = (size_t)(((p.rank + 7) & ~7) + 2 * NP * LN) * sizeof(float);
    if (smem > 48 * 1024) return PK_ERR_UNSUPPORTED;
    PK_LAUNCH_PDL((scan_rows_kernel<T, NP, LN>), grid, dim3(THREADS), smem, stream, p, seqs);
  }
  return PK_OK;
}

template <typename T>
int launch_scan(const PkSelectiveScan& p, const int4* seqs, int nseq, bool tiles, cudaStream_t stream) {
  if (p.N <= 4) return launch_scan<T, 4, 1>(p, seqs, nseq, tiles, stream);
  if (p.N <= 8) return launch_scan<T, 4, 2>(p, seqs, nseq, tiles, stream);
  if (p.N <= 16) return launch_scan<T, 4, 4>(p, seqs, nseq, tiles, stream);
  if (p.N <= 32) return launch_scan<T, 4, 8>(p, seqs, nseq, tiles, stream);
  if (p.N <= 64) return launch_scan<T, 4, 16>(p, seqs, nseq, tiles, stream);
  if (p.N <= 128) return launch_scan<T, 4, 32>(p, seqs, nseq, tiles, stream);
  if (p.N <= 256) return launch_scan<T, 8, 32>(p, seqs, nseq, tiles, stream);
  return PK_ERR_UNSUPPORTED;
}

template <typename T, int VW>
int launch_conv(const PkSelectiveScan& p, int rows, cudaStream_t stream) {
  const int blocks = (p.ldx + THREADS * VW - 1) / (THREADS * VW);
  int per = (int)((long long)rows * blocks / (148 * 16));
  per = per < 1 ? 1 : per > 32 ? 32 : per;
  const dim3 grid((rows + per - 1) / per, blocks);
  if (p.taps == 2) PK_LAUNCH_PDL((conv_kernel<T, 2, VW>), grid, dim3(THREADS), (size_t)0, stream, p, rows, per);
  else if (p.taps == 3) PK_LAUNCH_PDL((conv_kernel<T, 3, VW>), grid, dim3(THREADS), (size_t)0, stream, p, rows, per);
  else if (p.taps == 4) PK_LAUNCH_PDL((conv_kernel<T, 4, VW>), grid, dim3(THREADS), (size_t)0, stream, p, rows, per);
  else PK_LAUNCH_PDL((conv_kernel<T, 0, VW>), grid, dim3(THREADS), (size_t)0, stream, p, rows, per);
  return PK_OK;
}

template <typename T>
int launch_conv(const PkSelectiveScan& p, int rows, cudaStream_t stream) {
  const bool v4 = (p.inner & 3) == 0 && (p.ox & 3) == 0 && (p.ld & 3) == 0 && (p.ldx & 3) == 0 && ((uintptr_t)p.proj & 15) == 0 && ((uintptr_t)p.xc & 15) == 0 &&
                  ((uintptr_t)p.ring & 15) == 0 && ((uintptr_t)p.cb & 15) == 0;
  return v4 ? launch_conv<T, 4>(p, rows, stream) : launch_conv<T, 1>(p, rows, stream);
}

bool scan_ok(const PkSelectiveScan* d) {
  return d != nullptr && d->proj != nullptr && d->inner >= 1 && d->N >= 1 && d->rank >= 1 && d->taps >= 1 && d->xc != nullptr && d->ldx >= d->inner && d->pos != nullptr &&
         d->slot != nullptr && (d->taps == 1 || d->ring != nullptr) && d->ox >= 0 && d->oz >= 0 && d->ox + d->inner <= d->ld && d->oz + d->inner <= d->ld;
}

bool recurrence_ok(const PkSelectiveScan* d, const void* seqs, int nseq) {
  return scan_ok(d) && seqs != nullptr && nseq >= 1 && nseq <= 65535 && d->dbc != nullptr && d->ldb >= d->rank + 2 * d->N && d->dt_bias != nullptr && d->A != nullptr &&
         d->skip != nullptr && d->S != nullptr && d->out != nullptr && d->ldo >= d->inner &&
         ((d->N & 3) != 0 || (((uintptr_t)d->A & 15) == 0 && ((uintptr_t)d->S & 15) == 0));
}

}  // namespace

// Convolution and SiLU of all rows of a step -> xc.
PK_API int pk_scan_conv(const PkSelectiveScan* d, int rows, cudaStream_t stream) {
  if (!scan_ok(d) || d->cw == nullptr || d->cb == nullptr || rows < 1) return PK_ERR_BAD_ARG;
  return d->f32 ? launch_conv<float>(*d, rows, stream) : launch_conv<pk::bf16>(*d, rows, stream);
}

// d [rows, rank] (row stride ldd) -> out [rows, 2 kp] bf16, see split_kernel.
PK_API int pk_scan_split(const float* d, int ldd, int rank, int kp, int rows, void* out, cudaStream_t stream) {
  if (d == nullptr || out == nullptr || rank < 1 || kp < rank || ldd < rank || rows < 1) return PK_ERR_BAD_ARG;
  const long long n = ((long long)rows * kp + 255) / 256;
  PK_LAUNCH_PDL(split_kernel, dim3((unsigned)(n < 1184 ? n : 1184)), dim3(256), (size_t)0, stream, d, ldd, rank, kp, rows, (pk::bf16*)out);
  return PK_OK;
}

// Short portions: seqs [nseq] = {first row, tokens, slot, first position}. w_dt rows 16-byte aligned, ldw a multiple of 8.
PK_API int pk_scan_rows(const PkSelectiveScan* d, const void* seqs, int nseq, cudaStream_t stream) {
  if (!recurrence_ok(d, seqs, nseq) || d->w_dt == nullptr || d->ldw < ((d->rank + 7) & ~7) || (d->ldw & 7) != 0 || ((uintptr_t)d->w_dt & 15) != 0) return PK_ERR_BAD_ARG;
  return d->f32 ? launch_scan<float>(*d, (const int4*)seqs, nseq, false, stream) : launch_scan<pk::bf16>(*d, (const int4*)seqs, nseq, false, stream);
}

// Long portions, W_dt d given.
PK_API int pk_scan_tiles(const PkSelectiveScan* d, const void* seqs, int nseq, cudaStream_t stream) {
  if (!recurrence_ok(d, seqs, nseq) || d->dt == nullptr || d->ldt < d->inner) return PK_ERR_BAD_ARG;
  return d->f32 ? launch_scan<float>(*d, (const int4*)seqs, nseq, true, stream) : launch_scan<pk::bf16>(*d, (const int4*)seqs, nseq, true, stream);
}
