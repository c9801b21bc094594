// Selective scan of Mamba: per channel c and state n
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n,     y_c = sum_n S[c, n] C_n + D_c x_c,     out_c = y_c silu(z_c)
// with x behind a short causal convolution per channel and SiLU, dt_c = softplus(W_dt d + bias), and d, B, C from a product with x.
// State [slots, inner, state] fp32; the convolution's last inputs in a ring [slot][position modulo (taps - 1)][channel], as in the
// state space of ssd.cu: a token writes one entry, nothing shifts, inputs before position 0 are zero by position. Nothing is
// cleared on reuse of a slot: a portion that starts at position 0 starts from zero.
//
//   conv   x of all rows, into the type of the model (the operand of the product that yields d, B, C)
//   split  d as the sum of two bf16 terms side by side, so that W_dt d of many rows on the tensor cores keeps 16 bits of d
//   rows   portions of a few tokens: LN lanes per channel with NP states each, W_dt d in the same kernel (fp32 sums); a block takes a
//          few portions, which share its rows of W_dt
//   tiles  long portions: the same lanes walk the tokens in tiles of 8 to 32, two states per instruction. Between two barriers a block
//          requests tile i + 2 (cp.async), makes dt and dt x of tile i + 1, runs the recurrence over tile i, and gates and stores the
//          outputs of tile i - 1: independent work that fills the waits of the recurrence. The sums over a channel's lanes are taken for
//          LN tokens at a time (every exchange halves the number of partial sums)
// Everything but x and W_dt is fp32. A decay close to 1 that is rounded to fp32 is off by the same few 2^-25 at every step of a long
// memory; fp32 models therefore take what a state loses, exp(.) - 1, instead.
#include "../common/pk_vec.cuh"

// Plain data mirrored by the Python bindings.
struct PkSelectiveScan {
  const float* proj;       // [rows, ld]: x at column ox, z at oz
  const void* xc;          // [rows, ldx] x behind its convolution (model's type); conv writes it
  const float* dbc;        // [rows, ldb]: d, B at column oB, C at oC
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
  int ld, ox, oz, ldx, ldb, ldt, ldw, ldo, oB, oC, inner, N, rank, taps, f32;
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

template <int BYTES>
__device__ __forceinline__ void async_copy(void* dst, const void* src, int bytes) {      // the rest of BYTES is zero
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
  if (BYTES == 16) asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(src), "r"(bytes) : "memory");
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(a), "l"(src), "r"(bytes) : "memory");
}

// Block: THREADS / LN channels of up to SQ short portions.
template <typename T, int NP, int LN, int SQ>
__global__ void __launch_bounds__(THREADS, 4) scan_rows_kernel(const PkSelectiveScan p, const int4* seqs, int nseq) {
  constexpr int CB = THREADS / LN, NS = LN * NP, VE = 16 / sizeof(T), AHEAD = 4;
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, l = tid % LN, c = blockIdx.x * CB + tid / LN, n0 = l * NP;
  const bool live = c < p.inner;
  const int kw = (p.rank + 7) & ~7, unit = kw + 2 * NS;      // per portion: d [kw], B, C [NS]
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
  int4 sq[SQ];                                               // first row, tokens, slot, first position
  float s[SQ][NP];
  int most = 0;
#pragma unroll
  for (int q = 0; q < SQ; ++q) {
    const int at = blockIdx.y * SQ + q;
    sq[q] = at < nseq ? seqs[at] : make_int4(0, 0, 0, 0);
    most = max(most, sq[q].y);
#pragma unroll
    for (int k = 0; k < NP; ++k) s[q][k] = 0.f;
    if (live && sq[q].w > 0) load_states<NP>(p.S + ((size_t)sq[q].z * p.inner + c) * p.N, n0, p.N, s[q]);
  }
  const int dq = kw / 4, nq = dq + 2 * NS / 4;              // 16-byte pieces of a portion's d, and of d, B and C
  for (int t = 0; t < most; ++t) {
    // all of the tokens' loads are in flight together
    for (int e = tid; e < SQ * nq; e += THREADS) {
      int q = 0;
#pragma unroll
      for (int j = 1; j < SQ; ++j) q += e >= j * nq;
      int4 own = sq[0];
#pragma unroll
      for (int j = 1; j < SQ; ++j)
        if (q == j) own = sq[j];
      const int i = e - q * nq, part = i < dq ? 0 : i < dq + NS / 4 ? 1 : 2;
      const int k = (i - (part == 0 ? 0 : part == 1 ? dq : dq + NS / 4)) * 4, len = part == 0 ? p.rank : p.N;
      const bool in = t < own.y && k < len;
      const float* src = p.dbc + ((size_t)own.x + (in ? t : 0)) * p.ldb + (part == 0 ? 0 : part == 1 ? p.oB : p.oC) + (in ? k : 0);
      async_copy<16>(sm + q * unit + i * 4, src, in ? min(16, (len - k) * 4) : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    float x[SQ], z[SQ], in[SQ];
#pragma unroll
    for (int q = 0; q < SQ; ++q) {
      const bool on = t < sq[q].y && live;
      const size_t row = (size_t)sq[q].x + (on ? t : 0);
      const int col = live ? c : 0;
      x[q] = to_f<T>(((const T*)p.xc)[row * p.ldx + col]);
      z[q] = p.proj[row * p.ld + p.oz + col];
      in[q] = p.proj[row * p.ld + p.ox + col];
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float dot[SQ];
#pragma unroll
    for (int q = 0; q < SQ; ++q) dot[q] = 0.f;
    auto add = [&](const uint4& u, int k) {
      const T* e = reinterpret_cast<const T*>(&u);
#pragma unroll
      for (int i = 0; i < VE; i += 4)
#pragma unroll
        for (int q = 0; q < SQ; ++q) {
          const float4 d = *reinterpret_cast<const float4*>(sm + q * unit + k + i);
          dot[q] = fmaf(to_f<T>(e[i]), d.x, fmaf(to_f<T>(e[i + 1]), d.y, dot[q]));
          dot[q] = fmaf(to_f<T>(e[i + 2]), d.z, fmaf(to_f<T>(e[i + 3]), d.w, dot[q]));
        }
    };
    if (live) {
#pragma unroll
      for (int i = 0; i < AHEAD; ++i)
        if ((l + i * LN) * VE < kw) add(first[i], (l + i * LN) * VE);
#pragma unroll 2
      for (int k = (l + AHEAD * LN) * VE; k < kw; k += LN * VE) add(*reinterpret_cast<const uint4*>(wrow + k), k);
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1)
#pragma unroll
      for (int q = 0; q < SQ; ++q) dot[q] += __shfl_xor_sync(0xffffffffu, dot[q], o);
    float y[SQ];
#pragma unroll
    for (int q = 0; q < SQ; ++q) {      // a portion that has ended: dt 0 changes nothing
      const float* B = sm + q * unit + kw + n0;
      const float dt = t < sq[q].y ? softplus_series(dot[q] + bias) : 0.f, u = dt * x[q];
      y[q] = 0.f;
#pragma unroll
      for (int k = 0; k < NP; ++k) {
        s[q][k] = fmaf(u, B[k], decayed<T>(dt, a[k], s[q][k]));
        y[q] = fmaf(s[q][k], B[NS + k], y[q]);
      }
    }
#pragma unroll
    for (int o = LN / 2; o > 0; o >>= 1)
#pragma unroll
      for (int q = 0; q < SQ; ++q) y[q] += __shfl_xor_sync(0xffffffffu, y[q], o);
#pragma unroll
    for (int q = 0; q < SQ; ++q) {
      if (t >= sq[q].y) continue;
      T* out = (T*)p.out + ((size_t)sq[q].x + t) * p.ldo;
      if (live && l == 0) {
        out[c] = (T)(fmaf(skip, x[q], y[q]) * silu_of<T>(z[q]));
        if (sq[q].y - 1 - t < p.taps - 1) ring_at(p, sq[q].z, sq[q].w + t)[c] = in[q];
      }
      if (blockIdx.x == gridDim.x - 1)
        for (int i = p.inner + tid; i < p.ldo; i += THREADS) out[i] = (T)0.f;
    }
    if (t + 1 < most) __syncthreads();
  }
#pragma unroll
  for (int q = 0; q < SQ; ++q)
    if (live && sq[q].y > 0) store_states<NP>(p.S + ((size_t)sq[q].z * p.inner + c) * p.N, n0, p.N, s[q]);
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

typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float x, float y) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v)); }
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}

// What a lane needs of a token: dt, dt x, and B and C of its states.
template <int NP>
struct Token {
  float2 du;
  f32x2 B[NP / 2], C[NP / 2];
  __device__ __forceinline__ void load(const float2* d, const float* b, const float* c) {
    du = *d;
    if (NP == 2) {
      B[0] = *reinterpret_cast<const f32x2*>(b);
      C[0] = *reinterpret_cast<const f32x2*>(c);
      return;
    }
#pragma unroll
    for (int k = 0; k < NP / 4; ++k) {
      const ulonglong2 x = reinterpret_cast<const ulonglong2*>(b)[k], y = reinterpret_cast<const ulonglong2*>(c)[k];
      B[2 * k] = x.x;
      B[2 * k + 1] = x.y;
      C[2 * k] = y.x;
      C[2 * k + 1] = y.y;
    }
  }
};

// NP states of a channel over SUB tokens; y: what their lane adds to the outputs. Decays and inputs of all tokens come first, the
// serial part is one product per token.
template <typename T, int NP>
struct States {
  float a[NP], s[NP];
  f32x2 a2[NP / 2], s2[NP / 2];
  __device__ __forceinline__ void start() {
#pragma unroll
    for (int k = 0; k < NP / 2; ++k) {
      a2[k] = pack2(a[2 * k], a[2 * k + 1]);
      s2[k] = pack2(s[2 * k], s[2 * k + 1]);
    }
  }
  template <int SUB>
  __device__ __forceinline__ void run(const Token<NP> (&t)[SUB], float* y) {
    f32x2 e[SUB][NP / 2], in[SUB][NP / 2];
#pragma unroll
    for (int i = 0; i < SUB; ++i)
#pragma unroll
      for (int k = 0; k < NP / 2; ++k) {
        float x0, x1;
        unpack2(mul2(pack2(t[i].du.x, t[i].du.x), a2[k]), x0, x1);
        e[i][k] = sizeof(T) == 4 ? pack2(expm1f(x0), expm1f(x1)) : pack2(ex2(x0), ex2(x1));
        in[i][k] = mul2(pack2(t[i].du.y, t[i].du.y), t[i].B[k]);
      }
#pragma unroll
    for (int i = 0; i < SUB; ++i) {
      f32x2 sum = 0;
#pragma unroll
      for (int k = 0; k < NP / 2; ++k) {
        s2[k] = sizeof(T) == 4 ? fma2(pack2(1.f, 1.f), fma2(e[i][k], s2[k], s2[k]), in[i][k]) : fma2(e[i][k], s2[k], in[i][k]);
        sum = fma2(s2[k], t[i].C[k], sum);
      }
      float y0, y1;
      unpack2(sum, y0, y1);
      y[i] = y0 + y1;
    }
  }
  __device__ __forceinline__ void finish() {
#pragma unroll
    for (int k = 0; k < NP / 2; ++k) unpack2(s2[k], s[2 * k], s[2 * k + 1]);
  }
};

// Shared memory of a tiles block: STAGES raw tiles, then two tiles of (dt, dt x) and of sums.
template <typename T, int NP, int LN>
struct TileShape {
  static constexpr int CB = THREADS / LN, NS = LN * NP, TT = NS > 128 ? 8 : LN >= 8 && NS <= 32 ? 32 : 16, STAGES = 4;
  static constexpr int YS = CB + 8;                            // row of the sums: lanes of a group store to different banks
  static constexpr int DT = 0, Z = DT + TT * CB * 4, X = Z + TT * CB * 4, B = X + TT * CB * (int)sizeof(T), C = B + TT * NS * 4, RAW = C + TT * NS * 4;
  static constexpr int DU = STAGES * RAW, Y = DU + 2 * TT * CB * 8, BYTES = Y + 2 * TT * YS * 4;
};

// Block: THREADS / LN channels of one long portion, all its tokens.
template <typename T, int NP, int LN>
__global__ void __launch_bounds__(THREADS) scan_tiles_kernel(const PkSelectiveScan p, const int4* seqs) {
  pdl_trigger();
  pdl_wait();
  using Sh = TileShape<T, NP, LN>;
  constexpr int CB = Sh::CB, NS = Sh::NS, TT = Sh::TT, G = LN < TT ? LN : TT, QC = CB / 4, QN = NS / 4;
  extern __shared__ __align__(16) uint8_t smem[];
  const int4 sq = seqs[blockIdx.y];
  const int tid = threadIdx.x, l = tid % LN, ch = tid / LN, c0 = blockIdx.x * CB, c = c0 + ch, n0 = l * NP;
  const bool live = c < p.inner;
  const int n = sq.y, tiles = (n + TT - 1) / TT;
  States<T, NP> st;
#pragma unroll
  for (int k = 0; k < NP; ++k) st.a[k] = st.s[k] = 0.f;
  float* Sp = p.S + ((size_t)sq.z * p.inner + (live ? c : 0)) * p.N;
  if (live) {
    load_states<NP>(p.A + (size_t)c * p.N, n0, p.N, st.a);
    if (sq.w > 0) load_states<NP>(Sp, n0, p.N, st.s);
  }
  st.start();
  auto raw = [&](int i) { return smem + (i % Sh::STAGES) * Sh::RAW; };
  auto du = [&](int i) { return reinterpret_cast<float4*>(smem + Sh::DU) + (i & 1) * TT * CB / 2; };       // two channels per float4
  auto ys = [&](int i) { return reinterpret_cast<float*>(smem + Sh::Y) + (i & 1) * TT * Sh::YS; };
  auto request = [&](int i) {
    if (i < tiles) {
      uint8_t* dst = raw(i);
      for (int e = tid; e < TT * QC; e += THREADS) {
        const int t = i * TT + e / QC, cc = c0 + e % QC * 4;
        const bool in = t < n && cc < p.inner;
        const size_t row = (size_t)sq.x + (in ? t : 0);
        const int col = in ? cc : 0, bytes = in ? min(16, (p.inner - cc) * 4) : 0;
        async_copy<16>(dst + Sh::DT + e * 16, p.dt + row * p.ldt + col, bytes);
        async_copy<16>(dst + Sh::Z + e * 16, p.proj + row * p.ld + p.oz + col, bytes);
        async_copy<4 * sizeof(T)>(dst + Sh::X + e * 4 * sizeof(T), (const T*)p.xc + row * p.ldx + col, in ? 4 * (int)sizeof(T) : 0);
      }
      for (int e = tid; e < TT * QN; e += THREADS) {
        const int t = i * TT + e / QN, k = e % QN * 4;
        const bool in = t < n && k < p.N;
        const float* src = p.dbc + ((size_t)sq.x + (in ? t : 0)) * p.ldb;
        const int bytes = in ? min(16, (p.N - k) * 4) : 0;
        async_copy<16>(dst + Sh::B + e * 16, src + p.oB + (in ? k : 0), bytes);
        async_copy<16>(dst + Sh::C + e * 16, src + p.oC + (in ? k : 0), bytes);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto load_x = [&](const uint8_t* tile, int e, float (&x)[4]) { load_any<4>(tile + Sh::X, (size_t)e * 4, sizeof(T) == 4, x); };
  // a thread's groups of four channels have one place in a row
  float bias[4], skip[4];
  const int cq = c0 + tid % QC * 4;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    bias[k] = cq + k < p.inner ? p.dt_bias[cq + k] : 0.f;
    skip[k] = cq + k < p.inner ? p.skip[cq + k] : 0.f;
  }
  auto prepare = [&](int i) {                                 // dt and dt x; a token behind the end changes nothing
    const uint8_t* tile = raw(i);
    for (int e = tid; e < TT * QC; e += THREADS) {
      const float4 v = reinterpret_cast<const float4*>(tile + Sh::DT)[e];
      const float d[4] = {v.x, v.y, v.z, v.w};
      float x[4], dt[4];
      load_x(tile, e, x);
      const bool in = i * TT + e / QC < n;
#pragma unroll
      for (int k = 0; k < 4; ++k) dt[k] = in ? softplus_series(d[k] + bias[k]) : 0.f;
      du(i)[2 * e] = make_float4(dt[0], dt[0] * x[0], dt[1], dt[1] * x[1]);
      du(i)[2 * e + 1] = make_float4(dt[2], dt[2] * x[2], dt[3], dt[3] * x[3]);
    }
  };
  auto finish = [&](int i) {                                  // skip, gate, store, ring
    const uint8_t* tile = raw(i);
    for (int e = tid; e < TT * QC; e += THREADS) {
      const int t = i * TT + e / QC;
      if (t >= n || cq >= p.inner) continue;
      const float4 y4 = *reinterpret_cast<const float4*>(ys(i) + e / QC * Sh::YS + e % QC * 4), z4 = reinterpret_cast<const float4*>(tile + Sh::Z)[e];
      const float y[4] = {y4.x, y4.y, y4.z, y4.w}, z[4] = {z4.x, z4.y, z4.z, z4.w};
      float x[4], o[4];
      load_x(tile, e, x);
#pragma unroll
      for (int k = 0; k < 4; ++k) o[k] = fmaf(skip[k], x[k], y[k]) * silu_of<T>(z[k]);
      const size_t row = (size_t)sq.x + t;
      T* out = (T*)p.out + row * p.ldo + cq;
      if (cq + 4 <= p.inner) {
        store<4>(out, o);
      } else {
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (cq + k < p.inner) out[k] = (T)o[k];
      }
      if (n - 1 - t < p.taps - 1) {
        float* ring = ring_at(p, sq.z, sq.w + t) + cq;
        const float* in = p.proj + row * p.ld + p.ox + cq;
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (cq + k < p.inner) ring[k] = in[k];
      }
    }
    if (blockIdx.x == gridDim.x - 1 && p.ldo > p.inner) {
      const int pad = p.ldo - p.inner;
      for (int e = tid; e < TT * pad; e += THREADS)
        if (i * TT + e / pad < n) ((T*)p.out)[((size_t)sq.x + i * TT + e / pad) * p.ldo + p.inner + e % pad] = (T)0.f;
    }
  };
  request(0);
  request(1);
  asm volatile("cp.async.wait_group 1;" ::: "memory");
  __syncthreads();
  prepare(0);
  for (int i = 0; i < tiles; ++i) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                          // dt of tile i, sums of tile i - 1, raw tile i + 1; tile i - 2 is done with
    request(i + 2);
    if (i + 1 < tiles) prepare(i + 1);
    const float* B = reinterpret_cast<const float*>(raw(i) + Sh::B) + n0;
    const float* C = reinterpret_cast<const float*>(raw(i) + Sh::C) + n0;
    const float2* q = reinterpret_cast<const float2*>(du(i)) + ch;
    constexpr int SUB = NP > 4 ? 2 : 4;                       // tokens whose operands are in registers together
    Token<NP> tok[2][SUB];
    float y[TT];
    auto load = [&](int t) {
#pragma unroll
      for (int j = 0; j < SUB; ++j) tok[t / SUB & 1][j].load(q + (t + j) * CB, B + (t + j) * NS, C + (t + j) * NS);
    };
    load(0);
#pragma unroll
    for (int t = 0; t < TT; t += SUB) {
      if (t + SUB < TT) load(t + SUB);
      st.run(tok[t / SUB & 1], y + t);
    }
#pragma unroll
    for (int t = 0; t < TT; t += G) {
      float part[G];
#pragma unroll
      for (int j = 0; j < G; ++j) part[j] = y[t + j];
      float sum = group_sums<G>(part, l);
#pragma unroll
      for (int o = G; o < LN; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      y[t] = sum;
    }
    if (l < G) {
#pragma unroll
      for (int t = 0; t < TT; t += G) ys(i)[(t + l) * Sh::YS + ch] = y[t];
    }
    if (i > 0) finish(i - 1);
  }
  __syncthreads();
  finish(tiles - 1);
  st.finish();
  if (live) store_states<NP>(Sp, n0, p.N, st.s);
}

template <typename T, int NP, int LN, int SQ>
int launch_rows(const PkSelectiveScan& p, const int4* seqs, int nseq, cudaStream_t stream) {
  const size_t smem = (size_t)SQ * (((p.rank + 7) & ~7) + 2 * NP * LN) * sizeof(float);
  if (smem > 48 * 1024) return PK_ERR_UNSUPPORTED;
  const dim3 grid((p.inner + THREADS / LN - 1) / (THREADS / LN), (nseq + SQ - 1) / SQ);
  PK_LAUNCH_PDL((scan_rows_kernel<T, NP, LN, SQ>), grid, dim3(THREADS), smem, stream, p, seqs, nseq);
  return PK_OK;
}

template <typename T, int NP, int LN>
int launch_rows(const PkSelectiveScan& p, const int4* seqs, int nseq, cudaStream_t stream) {
  const bool fits = (size_t)4 * (((p.rank + 7) & ~7) + 2 * NP * LN) * sizeof(float) <= 48 * 1024;
  if (nseq == 1 || !fits) return launch_rows<T, NP, LN, 1>(p, seqs, nseq, stream);
  if (nseq <= 4) return launch_rows<T, NP, LN, 2>(p, seqs, nseq, stream);
  return launch_rows<T, NP, LN, 4>(p, seqs, nseq, stream);
}

template <typename T, int NP, int LN>
int launch_tiles(const PkSelectiveScan& p, const int4* seqs, int nseq, cudaStream_t stream) {
  using Sh = TileShape<T, NP, LN>;
  static PkDeviceOnce once;
  if (PkDeviceOnceGuard g{once}; g.needed()) {
    if (cudaFuncSetAttribute((const void*)scan_tiles_kernel<T, NP, LN>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sh::BYTES) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    g.done();
  }
  PK_LAUNCH_PDL((scan_tiles_kernel<T, NP, LN>), dim3((p.inner + Sh::CB - 1) / Sh::CB, nseq), dim3(THREADS), (size_t)Sh::BYTES, stream, p, seqs);
  return PK_OK;
}

template <typename T>
int launch_rows(const PkSelectiveScan& p, const int4* seqs, int nseq, cudaStream_t stream) {
  if (p.N <= 4) return launch_rows<T, 4, 1>(p, seqs, nseq, stream);
  if (p.N <= 8) return launch_rows<T, 4, 2>(p, seqs, nseq, stream);
  if (p.N <= 16) return launch_rows<T, 4, 4>(p, seqs, nseq, stream);
  if (p.N <= 32) return launch_rows<T, 4, 8>(p, seqs, nseq, stream);
  if (p.N <= 64) return launch_rows<T, 4, 16>(p, seqs, nseq, stream);
  if (p.N <= 128) return launch_rows<T, 4, 32>(p, seqs, nseq, stream);
  if (p.N <= 256) return launch_rows<T, 8, 32>(p, seqs, nseq, stream);
  return PK_ERR_UNSUPPORTED;
}

// Few states per thread: every scheduler needs several warps to fill the waits of a chain of tokens.
template <typename T>
int launch_tiles(const PkSelectiveScan& p, const int4* seqs, int nseq, cudaStream_t stream) {
  if (p.N <= 4) return launch_tiles<T, 2, 2>(p, seqs, nseq, stream);
  if (p.N <= 8) return launch_tiles<T, 2, 4>(p, seqs, nseq, stream);
  if (p.N <= 16) return launch_tiles<T, 2, 8>(p, seqs, nseq, stream);
  if (p.N <= 32) return launch_tiles<T, 4, 8>(p, seqs, nseq, stream);
  if (p.N <= 64) return launch_tiles<T, 4, 16>(p, seqs, nseq, stream);
  if (p.N <= 128) return launch_tiles<T, 4, 32>(p, seqs, nseq, stream);
  if (p.N <= 256) return launch_tiles<T, 8, 32>(p, seqs, nseq, stream);
  return PK_ERR_UNSUPPORTED;
}

template <typename T, int VW>
int launch_conv(const PkSelectiveScan& p, int rows, cudaStream_t stream) {
  const int blocks = (p.ldx + THREADS * VW - 1) / (THREADS * VW);
  int per = (int)((long long)rows * blocks / (148 * 16));
  const int least = rows < 64 ? 1 : 8;      // a block's first row fetches the whole window
  per = per < least ? least : per > 32 ? 32 : per;
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
  return scan_ok(d) && seqs != nullptr && nseq >= 1 && nseq <= 65535 && d->dbc != nullptr && d->oB >= d->rank && d->oC >= d->oB + d->N &&
         d->ldb >= d->oC + d->N && ((d->ldb | d->oB | d->oC) & 3) == 0 && ((uintptr_t)d->dbc & 15) == 0 && d->dt_bias != nullptr && d->A != nullptr &&
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

// Short portions: seqs [nseq] = {first row, tokens, slot, first position}. w_dt rows 16-byte aligned, ldw a multiple of 8; rows of dbc
// and the columns oB, oC start on 16 bytes.
PK_API int pk_scan_rows(const PkSelectiveScan* d, const void* seqs, int nseq, cudaStream_t stream) {
  if (!recurrence_ok(d, seqs, nseq) || d->w_dt == nullptr || d->ldw < ((d->rank + 7) & ~7) || (d->ldw & 7) != 0 || ((uintptr_t)d->w_dt & 15) != 0) return PK_ERR_BAD_ARG;
  return d->f32 ? launch_rows<float>(*d, (const int4*)seqs, nseq, stream) : launch_rows<pk::bf16>(*d, (const int4*)seqs, nseq, stream);
}

// Long portions, W_dt d given. Rows of dt, dbc and proj, and the columns oB, oC and oz, start on 16 bytes, rows of xc and out on four
// elements; xc is zero from inner on.
PK_API int pk_scan_tiles(const PkSelectiveScan* d, const void* seqs, int nseq, cudaStream_t stream) {
  if (!recurrence_ok(d, seqs, nseq) || d->dt == nullptr || d->ldt < d->inner) return PK_ERR_BAD_ARG;
  if (((d->ldt | d->ld | d->ldb | d->oB | d->oC | d->oz | d->ldx | d->ldo) & 3) != 0 || d->ldx < ((d->inner + 3) & ~3) || ((uintptr_t)d->dt & 15) != 0 ||
      ((uintptr_t)d->proj & 15) != 0 || ((uintptr_t)d->dbc & 15) != 0 || ((uintptr_t)d->xc & 15) != 0 || ((uintptr_t)d->out & 15) != 0)
    return PK_ERR_BAD_ARG;
  return d->f32 ? launch_tiles<float>(*d, (const int4*)seqs, nseq, stream) : launch_tiles<pk::bf16>(*d, (const int4*)seqs, nseq, stream);
}
