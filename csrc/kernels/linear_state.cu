// Recurrent mixers with an outer-product state: gated linear attention (a decay per key channel), the matrix memory of
// xLSTM (scalar gates with a running maximum), retention (a constant decay per head, rotated queries and keys), the state-space
// recurrence of Mamba-2 (a scalar decay per token and head) and HGRN2 (a forget gate per key channel which is also the key). All are
//   S_t = diag(a_t) S_{t-1} + b_t k_t v_t^T,    o_t = S_t^T q_t          S: [key dim, value dim], fp32
// with a_t a vector (GLA: a = sigmoid(z)^(1/tau), b = 1) or a scalar (mLSTM: a = exp(f + m_{t-1} - m_t), b = exp(i - m_t),
// m_t = max(f + m_{t-1}, i), m_0 = 0, and a normaliser n updated like a column of S with v = 1; retention: a = const, b = 1;
// state space: k = B, q = C, v = x, a = exp(A dt), b = dt, dt = softplus(z + bias), B and C shared by a group of heads, and
// o_t gets D x_t). The state-space inputs x, B and C pass a short causal convolution per channel and SiLU first; its last
// inputs are part of a request's state, a ring [slot][position modulo (taps - 1)][channel]. HGRN2: a = f = l + (1 - l) sigmoid(z +
// bias) with a lower bound l per channel, k = 1 - f, b = 1, q = silu(.).
// Everything here is fp32: gates, decays, states and products.
//
// State lives in slots [slot][head][key][value] so that requests of one batch keep theirs anywhere; a portion that starts
// at position 0 starts from zero whatever the slot holds. Two forms of one recurrence:
//   * rows (decode, portions of a few tokens): one block per (sequence, head, 32 value columns), the state slice in
//     registers, tokens in order;
//   * chunks of 64 tokens (prefill). The recurrence is linear in S, so only an elementwise scan over chunks is serial:
//       gates   per token: log decays (GLA; HGRN2's are made inside the next kernel), or log f, i and the running maximum m (mLSTM: an associative (+, max) scan)
//       intra   per (chunk, head): P_ij = sum_d q_i k_j exp(G_i - G_j) (j <= i), q~ = q exp(G_i), k~ = k exp(G_C - G_j)
//       kv      per (chunk, head, tile): k~^T V
//       scan    state before every chunk
//       out     per (chunk, head, tile): q~ S_c + P V
//     GLA's exponents are never split into exp(G_i) exp(-G_j) across a reference further away than the 16-token
//     sub-chunk between them: every factor is at most 1, whatever the decay. Retention takes the powers of its decays
//     from a table. The state space needs q k^T only once per group and takes its factors exp(G_i - G_j) dt_j, dt_j
//     exp(G_C - G_j) and exp(G_i) on the way into the products, where G is held as the sum of two floats.
// A last kernel normalises every head's output (after mLSTM's division by max(|n.q|, exp(-m)) + 1e-6), applies the output
// gate and writes the projection's input. Of the state space only the fp32 chunk form is here, its other kernels are in ssd.cu.
#include "../common/pk_rotary.cuh"
#include "../common/pk_state.cuh"

namespace {

using namespace pk;

enum { KIND_GLA = 0, KIND_MLSTM = 1, KIND_RETENTION = 2, KIND_SSD = 3, KIND_HGRN = 4 };
__host__ __device__ constexpr bool vector_decay(int kind) { return kind == KIND_GLA || kind == KIND_HGRN; }
constexpr int CH = 64;    // chunk
constexpr int SB = 16;    // sub-chunk

__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// HGRN2: the forget gate f of a channel and what it drops, 1 - f, each without a cancellation.
__device__ __forceinline__ void forget_gate(float z, float low, float& f, float& drop) {
  const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e / (1.f + e);
  f = low + (1.f - low) * (z >= 0.f ? big : small);
  drop = (1.f - low) * (z >= 0.f ? small : big);
}
__device__ __forceinline__ float log_forget(float f, float drop) { return f < 0.5f ? logf(fmaxf(f, 1e-37f)) : log1pf(-drop); }
__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// Columns of the fused input projection and the constants of one layer.
struct Mixer {
  const float* proj;   // [rows, ld]: q | k | v | gate | (i | f) or (low-rank decay input); HGRN2: q | f | v
  int ld;
  int oq, ok, ov, og, oi, of, oa;
  int H, D, V;
  float qscale;
  // mLSTM
  const float* bi;
  const float* bf;     // [H]; HGRN2: [H * D]
  float cap;
  // GLA
  const float* a2;     // [rank, H * D] (transposed low-rank up projection)
  const float* a2b;    // [H * D]
  int rank;
  float inv_tau;
  // retention
  const double* freq;  // [rot / 2] angular frequencies of the rotated leading part of queries and keys
  int rot;
  const float* pw;     // [H, 65] powers 0 .. 64 of every head's decay
  // state space: x (H x V) | B (groups x D) | C (groups x D) are columns ov .. of proj, dt columns odt .., the gate columns og ..
  const float* cw;     // [channels, taps] convolution, the last tap is the current token's
  const float* cb;     // [channels]
  const float* dtb;    // [H]
  const float* A;      // [H] negative
  const float* skip;   // [H]
  float* Cs;           // [slots, taps - 1, channels] last inputs of the convolution, by position modulo (taps - 1)
  int groups, taps, odt;
  // HGRN2
  const float* low;    // [H * D] lower bounds
  // state
  float* S;            // [slots, H, D, V]
  float* N;            // [slots, H, D]      (mLSTM)
  float* Ms;           // [slots, H]         (mLSTM)
};

// Outputs of the recurrence, before normalisation.
struct Raw {
  float* o;    // [rows, H, V]
  float* nq;   // [rows, H]   n . q       (mLSTM)
  float* m;    // [rows, H]   running max (mLSTM)
};

// ---------------------------------------------------------------------------------------
// rows form

constexpr int GR = 8;   // row groups (warps) of a block

template <int KIND, int RPT>
__global__ void __launch_bounds__(32 * GR) state_rows_kernel(const Mixer mx, const Raw raw, const int4* seqs) {
  pdl_trigger();
  pdl_wait();
  extern __shared__ float sm[];
  float* qs = sm;                 // [D]
  float* ks = qs + mx.D;          // [D]
  float* as = ks + mx.D;          // [D] (GLA)
  float* red = as + mx.D;         // [GR][33]
  __shared__ float s_sc[3];
  const int4 sq = seqs[blockIdx.z];          // first row, tokens, slot, first position
  const int h = blockIdx.y, lane = threadIdx.x & 31, g = threadIdx.x >> 5;
  const int D = mx.D, V = mx.V;
  const int col = blockIdx.x * 32 + lane;
  const bool is_v = col < V, is_n = KIND == KIND_MLSTM && col == V;
  const size_t head = (size_t)sq.z * mx.H + h;
  float* Sp = is_n ? mx.N + head * D : mx.S + head * D * V + col;
  const int st = is_n ? 1 : V;
  const bool live = is_v || is_n;
  float s[RPT];
#pragma unroll
  for (int j = 0; j < RPT; ++j) {
    const int d = g + j * GR;
    s[j] = live && d < D && sq.w > 0 ? Sp[(size_t)d * st] : 0.f;
  }
  float m_prev = KIND == KIND_MLSTM && sq.w > 0 ? mx.Ms[head] : 0.f;
  const float decay = KIND == KIND_RETENTION ? mx.pw[h * (CH + 1) + 1] : 0.f;
  for (int t = 0; t < sq.y; ++t) {
    const float* pr = mx.proj + (size_t)(sq.x + t) * mx.ld;
    if (KIND == KIND_RETENTION) {
      // one item per rotated pair, then one per channel that passes
      const int half = mx.rot / 2;
      const float* q = pr + mx.oq + h * D;
      const float* k = pr + mx.ok + h * D;
      for (int i = threadIdx.x; i < D - half; i += 32 * GR) {
        if (i < half) {
          float s, c, qu = q[i] * mx.qscale, qv = q[i + half] * mx.qscale, ku = k[i], kv = k[i + half];
          rotary_sincos(mx.freq[i], sq.w + t, s, c);
          rotate_pair(qu, qv, s, c);
          rotate_pair(ku, kv, s, c);
          qs[i] = qu;
          qs[i + half] = qv;
          ks[i] = ku;
          ks[i + half] = kv;
        } else {
          qs[i + half] = q[i + half] * mx.qscale;
          ks[i + half] = k[i + half];
        }
      }
    } else if (KIND == KIND_HGRN) {
      for (int d = threadIdx.x; d < D; d += 32 * GR) {
        qs[d] = silu_exact(pr[mx.oq + h * D + d]);
        float f;
        forget_gate(pr[mx.of + h * D + d] + mx.bf[h * D + d], mx.low[h * D + d], f, ks[d]);
      }
    } else {
      for (int d = threadIdx.x; d < D; d += 32 * GR) {
        qs[d] = pr[mx.oq + h * D + d] * mx.qscale;
        ks[d] = pr[mx.ok + h * D + d];
        if (KIND == KIND_GLA) {
          float z = mx.a2b[h * D + d];
          for (int r = 0; r < mx.rank; ++r) z = fmaf(mx.a2[(size_t)r * mx.H * D + h * D + d], pr[mx.oa + r], z);
          as[d] = expf(log_sigmoid(z) * mx.inv_tau);
        }
      }
    }
    if (KIND == KIND_MLSTM) {
      const float gi = soft_cap(pr[mx.oi + h] + mx.bi[h], mx.cap);
      const float gf = log_sigmoid(soft_cap(pr[mx.of + h] + mx.bf[h], mx.cap));
      const float m = fmaxf(gf + m_prev, gi);
      if (threadIdx.x == 0) {
        s_sc[0] = expf(gf + m_prev - m);
        s_sc[1] = expf(gi - m);
        if (blockIdx.x == 0) raw.m[(size_t)(sq.x + t) * mx.H + h] = m;
      }
      m_prev = m;
    }
    float v = is_v ? pr[mx.ov + h * V + col] : (is_n ? 1.f : 0.f);
    __syncthreads();
    float part = 0.f;
    if (!vector_decay(KIND)) {
      const float a = KIND == KIND_MLSTM ? s_sc[0] : decay;
      if (KIND == KIND_MLSTM) v *= s_sc[1];
#pragma unroll
      for (int j = 0; j < RPT; ++j) {
        const int d = g + j * GR;
        if (d < D) {
          s[j] = fmaf(a, s[j], ks[d] * v);
          part = fmaf(s[j], qs[d], part);
        }
      }
    } else {
#pragma unroll
      for (int j = 0; j < RPT; ++j) {
        const int d = g + j * GR;
        if (d < D) {
          // HGRN2: what is dropped is replaced, which keeps the sum's digits when f is close to 1
          s[j] = KIND == KIND_HGRN ? fmaf(ks[d], v - s[j], s[j]) : fmaf(as[d], s[j], ks[d] * v);
          part = fmaf(s[j], qs[d], part);
        }
      }
    }
    red[g * 33 + lane] = part;
    __syncthreads();
    if (g == 0 && live) {
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < GR; ++i) o += red[i * 33 + lane];
      if (is_n) raw.nq[(size_t)(sq.x + t) * mx.H + h] = o;
      else raw.o[((size_t)(sq.x + t) * mx.H + h) * V + col] = o;
    }
    __syncthreads();
  }
  if (live) {
#pragma unroll
    for (int j = 0; j < RPT; ++j) {
      const int d = g + j * GR;
      if (d < D) Sp[(size_t)d * st] = s[j];
    }
  }
}

// ---------------------------------------------------------------------------------------
// chunk form

// {first row, tokens, slot, first position} per sequence; {first row, tokens, sequence, chunk of the sequence} per chunk;
// chunk0[sequence] = index of its first chunk
struct Chunks {
  const int4* seqs;
  const int4* chunks;
  const int* chunk0;
  int nseq, nchunks;
};

struct Work {
  float* logd;   // GLA: [long rows, H * D] log decays, indexed by chunk * 64 + i
  float* lf;     // mLSTM: [chunk * 64 + i, H]
  float* ig;
  float* qt;     // [chunk, H, 64, D]  q exp(G_i)
  float* kt;     // [chunk, H, 64, D]  k exp(G_C - G_j)
  float* dec;    // [chunk, H, D]      exp(G_C)
  float* P;      // [chunk, H, 64, 64]
  float* KV;     // [chunk, H, D, V]   k~^T V, then the state before the chunk
  float* NK;     // [chunk, H, D]      sum_j k~_j, then n before the chunk (mLSTM)
  float* xbc;    // state space: [chunk * 64 + i, channels] x | B | C behind the convolution
  float* dt;     // state space: [chunk, H, 64] step sizes
  float2* G;     // state space: [chunk, H, 64] running log decay, high and low part
  int dec_w;     // entries of dec per chunk and head: D, or 1 (one decay for all channels)
};

// GLA: log decay of every channel, z = a2 (a1 h) + bias. One block per (chunk, 8 rows of it), channels over the threads.
__global__ void __launch_bounds__(256) gla_gates_kernel(const Mixer mx, const Chunks ck, const Work wk) {
  extern __shared__ float sm[];   // [8][rank]
  const int4 c = ck.chunks[blockIdx.x];
  const int r0 = blockIdx.y * 8;
  for (int i = threadIdx.x; i < 8 * mx.rank; i += 256) {
    const int r = i / mx.rank, j = i - r * mx.rank;
    sm[i] = r0 + r < c.y ? mx.proj[(size_t)(c.x + r0 + r) * mx.ld + mx.oa + j] : 0.f;
  }
  __syncthreads();
  const int HD = mx.H * mx.D;
  for (int ch = blockIdx.z * 256 + threadIdx.x; ch < HD; ch += 256 * gridDim.z) {
    float z[8];
#pragma unroll
    for (int r = 0; r < 8; ++r) z[r] = mx.a2b[ch];
    for (int j = 0; j < mx.rank; ++j) {
      const float w = mx.a2[(size_t)j * HD + ch];
#pragma unroll
      for (int r = 0; r < 8; ++r) z[r] = fmaf(w, sm[r * mx.rank + j], z[r]);
    }
#pragma unroll
    for (int r = 0; r < 8; ++r)
      if (r0 + r < CH) wk.logd[((size_t)blockIdx.x * CH + r0 + r) * HD + ch] = r0 + r < c.y ? log_sigmoid(z[r]) * mx.inv_tau : 0.f;
  }
}

// mLSTM: log f, i and the running maximum of every token of a portion. m_t = max(a + m_0, b) with (a, b) the running
// composition of (f_t, i_t): (a1, b1) then (a2, b2) = (a1 + a2, max(b1 + a2, b2)). One block per (sequence, head).
__global__ void __launch_bounds__(256) mlstm_gates_kernel(const Mixer mx, const Raw raw, const Chunks ck, const Work wk) {
  __shared__ float wa[8], wb[8], s_m;
  const int4 sq = ck.seqs[blockIdx.x];
  const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, w = tid >> 5;
  if (tid == 0) s_m = sq.w > 0 ? mx.Ms[(size_t)sq.z * mx.H + h] : 0.f;
  __syncthreads();
  const size_t base = (size_t)ck.chunk0[blockIdx.x] * CH;
  for (int t0 = 0; t0 < sq.y; t0 += 256) {
    const int t = t0 + tid;
    float a = 0.f, b = -INFINITY;
    if (t < sq.y) {
      const float* pr = mx.proj + (size_t)(sq.x + t) * mx.ld;
      b = soft_cap(pr[mx.oi + h] + mx.bi[h], mx.cap);
      a = log_sigmoid(soft_cap(pr[mx.of + h] + mx.bf[h], mx.cap));
      wk.lf[(base + t) * mx.H + h] = a;
      wk.ig[(base + t) * mx.H + h] = b;
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, a, o), pb = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) {
        b = fmaxf(pb + a, b);
        a += pa;
      }
    }
    if (lane == 31) { wa[w] = a; wb[w] = b; }
    __syncthreads();
    float m = s_m;
    for (int i = 0; i < w; ++i) m = fmaxf(wa[i] + m, wb[i]);
    m = fmaxf(a + m, b);
    if (t < sq.y) raw.m[(size_t)(sq.x + t) * mx.H + h] = m;
    __syncthreads();
    if (tid == 255) s_m = m;
    __syncthreads();
  }
}

// mLSTM intra-chunk part. One block per (chunk, head).
__global__ void __launch_bounds__(256) mlstm_intra_kernel(const Mixer mx, const Raw raw, const Chunks ck, const Work wk) {
  __shared__ float Qs[32][CH + 4], Ks[32][CH + 4];
  __shared__ double Fd[CH];
  __shared__ float ig[CH], mi[CH], eq[CH], ek[CH];
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int4 cd = ck.chunks[c];
  const int len = cd.y, D = mx.D;
  const size_t ch = (size_t)c * mx.H + h;
  if (tid < CH) {
    ig[tid] = tid < len ? wk.ig[((size_t)c * CH + tid) * mx.H + h] : 0.f;
    mi[tid] = tid < len ? raw.m[(size_t)(cd.x + tid) * mx.H + h] : 0.f;
  }
  if (tid == 0) {
    double f = 0.0;
    for (int i = 0; i < CH; ++i) {
      f += i < len ? (double)wk.lf[((size_t)c * CH + i) * mx.H + h] : 0.0;
      Fd[i] = f;
    }
  }
  __syncthreads();
  const int4 sq = ck.seqs[cd.z];
  const float m_start = cd.w > 0 ? raw.m[(size_t)(cd.x - 1) * mx.H + h] : (sq.w > 0 ? mx.Ms[(size_t)sq.z * mx.H + h] : 0.f);
  const float m_end = mi[len - 1];
  const double F_end = Fd[len - 1];
  if (tid < CH) {
    eq[tid] = tid < len ? expf((float)(Fd[tid] + (double)m_start - (double)mi[tid])) : 0.f;
    ek[tid] = tid < len ? expf((float)(F_end - Fd[tid] + (double)ig[tid] - (double)m_end)) : 0.f;
  }
  const float dec = expf((float)(F_end + (double)m_start - (double)m_end));
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int d0 = 0; d0 < D; d0 += 32) {
    for (int i = tid; i < CH * 32; i += 256) {
      const int r = i >> 5, d = i & 31;
      float q = 0.f, k = 0.f;
      if (d0 + d < D) {
        if (r < len) {
          const float* pr = mx.proj + (size_t)(cd.x + r) * mx.ld + h * D + d0 + d;
          q = pr[mx.oq] * mx.qscale;
          k = pr[mx.ok];
        }
        wk.qt[(ch * CH + r) * D + d0 + d] = q * eq[r];
        wk.kt[(ch * CH + r) * D + d0 + d] = k * ek[r];
        if (r == 0) wk.dec[ch * D + d0 + d] = dec;
      }
      Qs[d][r] = q;
      Ks[d][r] = k;
    }
    __syncthreads();
#pragma unroll 8
    for (int d = 0; d < 32; ++d) {
      const float4 a = *reinterpret_cast<const float4*>(&Qs[d][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Ks[d][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    float4 out;
    float* ov = reinterpret_cast<float*>(&out);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = tx * 4 + j;
      ov[j] = s <= r && r < len ? acc[i][j] * expf((float)(Fd[r] - Fd[s]) + (ig[s] - mi[r])) : 0.f;
    }
    *reinterpret_cast<float4*>(wk.P + (ch * CH + r) * CH + tx * 4) = out;
  }
}

// Retention intra-chunk part. One block per (chunk, head). Channels are walked so that both halves of a rotated pair are
// neighbours: c < rot is half (c & 1) of pair c / 2, the others follow unchanged.
__global__ void __launch_bounds__(256) retention_intra_kernel(const Mixer mx, const Chunks ck, const Work wk) {
  __shared__ float Qs[32][CH + 4], Ks[32][CH + 4];
  __shared__ float pw[CH + 1];
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int4 cd = ck.chunks[c];
  const int len = cd.y, D = mx.D, half = mx.rot / 2;
  const int4 sq = ck.seqs[cd.z];
  const int pos0 = sq.w + cd.x - sq.x;
  const size_t ch = (size_t)c * mx.H + h;
  if (tid <= CH) pw[tid] = mx.pw[h * (CH + 1) + tid];
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int c0 = 0; c0 < D; c0 += 32) {
    for (int i = tid; i < CH * 16; i += 256) {
      const int r = i >> 4, x = (i & 15) * 2, cc = c0 + x;
      const bool turn = cc < mx.rot;
      const int d0 = turn ? cc >> 1 : cc, d1 = turn ? d0 + half : cc + 1;
      float qu = 0.f, qv = 0.f, ku = 0.f, kv = 0.f;
      if (cc < D && r < len) {
        const float* pr = mx.proj + (size_t)(cd.x + r) * mx.ld + h * D;
        qu = pr[mx.oq + d0] * mx.qscale;
        ku = pr[mx.ok + d0];
        if (d1 < D) {
          qv = pr[mx.oq + d1] * mx.qscale;
          kv = pr[mx.ok + d1];
        }
        if (turn) {
          float s, co;
          rotary_sincos(mx.freq[d0], pos0 + r, s, co);
          rotate_pair(qu, qv, s, co);
          rotate_pair(ku, kv, s, co);
        }
      }
      if (cc < D) {
        const float eq = r < len ? pw[r + 1] : 0.f, ek = r < len ? pw[len - 1 - r] : 0.f;
        float* qt = wk.qt + (ch * CH + r) * D;
        float* kt = wk.kt + (ch * CH + r) * D;
        qt[d0] = qu * eq;
        kt[d0] = ku * ek;
        if (d1 < D) {
          qt[d1] = qv * eq;
          kt[d1] = kv * ek;
        }
        if (r == 0) {
          wk.dec[ch * D + d0] = pw[len];
          if (d1 < D) wk.dec[ch * D + d1] = pw[len];
        }
      }
      Qs[x][r] = qu;
      Qs[x + 1][r] = qv;
      Ks[x][r] = ku;
      Ks[x + 1][r] = kv;
    }
    __syncthreads();
#pragma unroll 8
    for (int d = 0; d < 32; ++d) {
      const float4 a = *reinterpret_cast<const float4*>(&Qs[d][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Ks[d][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    float4 out;
    float* ov = reinterpret_cast<float*>(&out);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = tx * 4 + j;
      ov[j] = s <= r && r < len ? acc[i][j] * pw[r - s] : 0.f;
    }
    *reinterpret_cast<float4*>(wk.P + (ch * CH + r) * CH + tx * 4) = out;
  }
}

// State space, what enters the recurrence: blocks (chunk, y) convolve 256 channels each; the blocks behind them take 8 heads
// each, one warp per head: step sizes, running log decay over the chunk (summed in double precision), decay of the chunk.
template <int TAPS>      // 0: any number
__global__ void __launch_bounds__(256) ssd_inputs_kernel(const Mixer mx, const Chunks ck, const Work wk, int conv_blocks) {
  const int c = blockIdx.x, tid = threadIdx.x;
  const int4 cd = ck.chunks[c], sq = ck.seqs[cd.z];
  const int t0 = cd.x - sq.x, pos0 = sq.w + t0;      // first token of the chunk
  if ((int)blockIdx.y < conv_blocks) {
    const int CD = ssd_channels(mx), ch = blockIdx.y * 256 + tid;
    if (ch >= CD) return;
    float* out = wk.xbc + (size_t)c * CH * CD + ch;
    conv_silu_rows<TAPS>(mx, sq.z, cd.x, t0, pos0, cd.y, ch, [&](int r, float y) { out[(size_t)r * CD] = y; });
    return;
  }
  const int h = (blockIdx.y - conv_blocks) * 8 + (tid >> 5), lane = tid & 31;
  if (h >= mx.H) return;
  const size_t ch = (size_t)c * mx.H + h;
  float total;
  ssd_decays<CH / 32>(mx, cd.x, cd.y, h, lane, wk.dt + ch * CH, wk.G + ch * CH, &total);
  if (lane == 31) wk.dec[ch] = expf(total);
}

// P_ij = C_i . B_j of a (chunk, group of heads).
__global__ void __launch_bounds__(256) ssd_scores_kernel(const Mixer mx, const Chunks ck, const Work wk) {
  __shared__ float Qs[32][CH + 4], Ks[32][CH + 4];
  const int c = blockIdx.x, g = blockIdx.y, tid = threadIdx.x;
  const int len = ck.chunks[c].y, D = mx.D, CD = ssd_channels(mx);
  const float* kb = wk.xbc + (size_t)c * CH * CD + mx.H * mx.V + g * D;
  const float* qb = kb + mx.groups * D;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int d0 = 0; d0 < D; d0 += 32) {
    for (int i = tid; i < CH * 32; i += 256) {
      const int r = i >> 5, d = i & 31;
      const bool in = r < len && d0 + d < D;
      Qs[d][r] = in ? qb[(size_t)r * CD + d0 + d] : 0.f;
      Ks[d][r] = in ? kb[(size_t)r * CD + d0 + d] : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int d = 0; d < 32; ++d) {
      const float4 a = *reinterpret_cast<const float4*>(&Qs[d][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Ks[d][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
    *reinterpret_cast<float4*>(wk.P + (((size_t)c * mx.groups + g) * CH + ty * 4 + i) * CH + tx * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
}

// Intra-chunk part of GLA and HGRN2. One block per (chunk, head); 32 channels at a time. Thread (ti, tj) owns the entries
// (16 a + ti, 16 b + tj) for all sub-chunk pairs b <= a.
template <int KIND>
__global__ void __launch_bounds__(256) gla_intra_kernel(const Mixer mx, const Chunks ck, const Work wk) {
  constexpr int DT = 32, LD = DT + 1;
  __shared__ float q[CH][LD], k[CH][LD], g[CH][LD];     // g: running log decay inside the sub-chunk
  __shared__ float qd[CH][LD], kd[CH][LD];              // q exp(g), k exp(total - g)
  __shared__ float tot[CH / SB][DT];
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int4 cd = ck.chunks[c];
  const int len = cd.y, D = mx.D, HD = mx.H * D;
  const size_t ch = (size_t)c * mx.H + h;
  const int tj = tid & 15, ti = tid >> 4;
  float dg[4] = {0.f, 0.f, 0.f, 0.f};
  float od[6] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f};   // (1,0) (2,1) (3,2) (2,0) (3,1) (3,0)
  for (int d0 = 0; d0 < D; d0 += DT) {
    const int nd = min(DT, D - d0);
    for (int i = tid; i < CH * DT; i += 256) {
      const int r = i >> 5, d = i & 31;
      float qv = 0.f, kv = 0.f, lv = 0.f;
      if (d < nd && r < len) {
        const float* pr = mx.proj + (size_t)(cd.x + r) * mx.ld + h * D + d0 + d;
        if (KIND == KIND_HGRN) {
          float f;
          qv = silu_exact(pr[mx.oq]);
          forget_gate(pr[mx.of] + mx.bf[h * D + d0 + d], mx.low[h * D + d0 + d], f, kv);
          lv = log_forget(f, kv);
        } else {
          qv = pr[mx.oq] * mx.qscale;
          kv = pr[mx.ok];
          lv = wk.logd[((size_t)c * CH + r) * HD + h * D + d0 + d];
        }
      }
      q[r][d] = qv;
      k[r][d] = kv;
      g[r][d] = lv;
    }
    __syncthreads();
    if (tid < 128) {
      const int d = tid & 31, a = tid >> 5;
      float s = 0.f;
#pragma unroll
      for (int r = 0; r < SB; ++r) {
        s += g[a * SB + r][d];
        g[a * SB + r][d] = s;
      }
      tot[a][d] = s;
    }
    __syncthreads();
    for (int i = tid; i < CH * DT; i += 256) {
      const int r = i >> 5, d = i & 31, a = r >> 4;
      const float e1 = expf(g[r][d]), e2 = expf(tot[a][d] - g[r][d]);
      const float qv = q[r][d] * e1, kv = k[r][d] * e2;
      qd[r][d] = qv;
      kd[r][d] = kv;
      if (d < nd) {
        float pre = 0.f, suf = 0.f;
        for (int b = 0; b < CH / SB; ++b) {
          if (b < a) pre += tot[b][d];
          if (b > a) suf += tot[b][d];
        }
        wk.qt[(ch * CH + r) * D + d0 + d] = qv * expf(pre);
        wk.kt[(ch * CH + r) * D + d0 + d] = kv * expf(suf);
        if (r == 0) wk.dec[ch * D + d0 + d] = expf(tot[0][d] + tot[1][d] + tot[2][d] + tot[3][d]);
      }
    }
    __syncthreads();
    for (int d = 0; d < nd; ++d) {
      const float e1 = expf(tot[1][d]), e2 = expf(tot[2][d]);
      const float q1 = qd[SB + ti][d], q2 = qd[2 * SB + ti][d], q3 = qd[3 * SB + ti][d];
      const float k0 = kd[tj][d], k1 = kd[SB + tj][d], k2 = kd[2 * SB + tj][d];
      od[0] = fmaf(q1, k0, od[0]);
      od[1] = fmaf(q2, k1, od[1]);
      od[2] = fmaf(q3, k2, od[2]);
      od[3] = fmaf(q2 * e1, k0, od[3]);
      od[4] = fmaf(q3 * e2, k1, od[4]);
      od[5] = fmaf(q3 * e2 * e1, k0, od[5]);
      if (tj <= ti) {
#pragma unroll
        for (int a = 0; a < 4; ++a)
          dg[a] = fmaf(q[a * SB + ti][d] * k[a * SB + tj][d], expf(g[a * SB + ti][d] - g[a * SB + tj][d]), dg[a]);
      }
    }
    __syncthreads();
  }
  float* P = wk.P + ch * CH * CH;
#pragma unroll
  for (int a = 0; a < 4; ++a) {
#pragma unroll
    for (int b = 0; b < 4; ++b) {
      float v = 0.f;
      if (a == b) v = tj <= ti ? dg[a] : 0.f;
      else if (a == b + 1) v = od[b];
      else if (a == b + 2) v = od[3 + b];
      else if (a == b + 3) v = od[5];
      P[(a * SB + ti) * CH + b * SB + tj] = v;
    }
  }
}

// KV = k~^T V for one chunk, head and 64 x 64 tile of the state; mLSTM's first value tile also sums k~ over the chunk.
template <bool SSD>
__global__ void __launch_bounds__(256) chunk_kv_kernel(const Mixer mx, const Chunks ck, const Work wk, int dtiles) {
  __shared__ float Ks[CH][64 + 4], Vs[CH][64 + 4];
  const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int d0 = (blockIdx.z % dtiles) * 64, v0 = (blockIdx.z / dtiles) * 64;
  const int4 cd = ck.chunks[c];
  const int D = mx.D, V = mx.V;
  const size_t ch = (size_t)c * mx.H + h;
  if (SSD) {
    __shared__ float w[CH];
    const int CD = ssd_channels(mx);
    if (tid < CH) {
      const float2 g = wk.G[ch * CH + tid], e = wk.G[ch * CH + CH - 1];
      w[tid] = tid < cd.y ? wk.dt[ch * CH + tid] * expf((e.x - g.x) + (e.y - g.y)) : 0.f;
    }
    __syncthreads();
    const float* row = wk.xbc + (size_t)c * CH * CD;
    const int b0 = mx.H * V + h / (mx.H / mx.groups) * D;
    for (int i = tid; i < CH * 64; i += 256) {
      const int r = i >> 6, x = i & 63;
      const bool in = r < cd.y;
      Ks[r][x] = in && d0 + x < D ? row[(size_t)r * CD + b0 + d0 + x] : 0.f;
      Vs[r][x] = in && v0 + x < V ? row[(size_t)r * CD + h * V + v0 + x] * w[r] : 0.f;
    }
  } else
  for (int i = tid; i < CH * 64; i += 256) {
    const int r = i >> 6, x = i & 63;
    Ks[r][x] = d0 + x < D ? wk.kt[(ch * CH + r) * D + d0 + x] : 0.f;
    Vs[r][x] = v0 + x < V && r < cd.y ? mx.proj[(size_t)(cd.x + r) * mx.ld + mx.ov + h * V + v0 + x] : 0.f;
  }
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 8
  for (int r = 0; r < CH; ++r) {
    const float4 a = *reinterpret_cast<const float4*>(&Ks[r][ty * 4]);
    const float4 b = *reinterpret_cast<const float4*>(&Vs[r][tx * 4]);
    const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int d = d0 + ty * 4 + i;
    if (d >= D) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int v = v0 + tx * 4 + j;
      if (v < V) wk.KV[(ch * D + d) * V + v] = acc[i][j];
    }
  }
  if (wk.NK != nullptr && v0 == 0 && tid < 64 && d0 + tid < D) {
    float s = 0.f;
    for (int r = 0; r < CH; ++r) s += Ks[r][tid];
    wk.NK[ch * D + d0 + tid] = s;
  }
}

// Serial over the chunks of a sequence, one thread per VW adjacent state elements: KV[c] <- state before chunk c, slot <-
// final state.
template <int VW>
__global__ void __launch_bounds__(256) chunk_scan_kernel(const Mixer mx, const Chunks ck, const Work wk) {
  const int4 sq = ck.seqs[blockIdx.z];
  const int h = blockIdx.y, D = mx.D, V = mx.V;
  const int g = blockIdx.x * 256 + threadIdx.x;      // group of [D, V / VW], then element of [D]
  const int groups = D * V / VW;
  if (g >= groups + (wk.NK != nullptr ? D : 0)) return;
  const bool is_n = g >= groups;
  const int d = is_n ? g - groups : g * VW / V;
  const int c0 = ck.chunk0[blockIdx.z], n = (sq.y + CH - 1) / CH;
  const size_t head = (size_t)sq.z * mx.H + h;
  float* state = is_n ? mx.N + head * D + d : mx.S + head * D * V + (size_t)g * VW;
  float* kv = is_n ? wk.NK + ((size_t)c0 * mx.H + h) * D + d : wk.KV + ((size_t)c0 * mx.H + h) * D * V + (size_t)g * VW;
  const float* dec = wk.dec + ((size_t)c0 * mx.H + h) * wk.dec_w + (wk.dec_w > 1 ? d : 0);
  const size_t kv_step = (size_t)mx.H * D * (is_n ? 1 : V), dec_step = (size_t)mx.H * wk.dec_w;
  auto load = [&](const float* p) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (VW == 4 && !is_n) v = *reinterpret_cast<const float4*>(p);
    else v.x = *p;
    return v;
  };
  auto store = [&](float* p, const float4& v) {
    if (VW == 4 && !is_n) *reinterpret_cast<float4*>(p) = v;
    else *p = v.x;
  };
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (sq.w > 0) s = load(state);
  constexpr int AHEAD = 8;      // chunks whose loads are in flight together: only the fma chain is serial
  for (int c = 0; c < n; c += AHEAD) {
    float4 add[AHEAD];
    float dc[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c + i < n) {
        add[i] = load(kv + (size_t)(c + i) * kv_step);
        dc[i] = dec[(size_t)(c + i) * dec_step];
      }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c + i < n) {
        store(kv + (size_t)(c + i) * kv_step, s);
        s.x = fmaf(dc[i], s.x, add[i].x);
        s.y = fmaf(dc[i], s.y, add[i].y);
        s.z = fmaf(dc[i], s.z, add[i].z);
        s.w = fmaf(dc[i], s.w, add[i].w);
      }
  }
  store(state, s);
}

// o = q~ S_c + P V for one chunk, head and 64 value columns.
template <bool SSD>
__global__ void __launch_bounds__(256) chunk_out_kernel(const Mixer mx, const Raw raw, const Chunks ck, const Work wk) {
  __shared__ float As[32][CH + 4], Bs[32][64 + 4];
  const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * 64, tid = threadIdx.x;
  const int4 cd = ck.chunks[c];
  const int D = mx.D, V = mx.V;
  const size_t ch = (size_t)c * mx.H + h;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // state space: rows of x and C, exp(G_i), running decays and steps of the chunk
  __shared__ float eg[CH], dts[CH];
  __shared__ float2 gs[CH];
  const int CD = SSD ? ssd_channels(mx) : 0, group = SSD ? h / (mx.H / mx.groups) : 0;
  const float* xrow = SSD ? wk.xbc + (size_t)c * CH * CD : nullptr;
  const float* crow = SSD ? xrow + mx.H * V + (mx.groups + group) * D : nullptr;
  const float* cb = SSD ? wk.P + ((size_t)c * mx.groups + group) * CH * CH : nullptr;
  if (SSD) {
    if (tid < CH) {
      const float2 g = wk.G[ch * CH + tid];
      gs[tid] = g;
      eg[tid] = expf(g.x + g.y);
      dts[tid] = wk.dt[ch * CH + tid];
    }
    __syncthreads();
  }
  float nq = 0.f;     // mLSTM, value tile 0: thread tid < 64 owns row tid
  const bool want_n = wk.NK != nullptr && blockIdx.z == 0 && tid < CH;
  const int steps_d = (D + 31) / 32, steps = steps_d + CH / 32;
  for (int s = 0; s < steps; ++s) {
    const bool inter = s < steps_d;
    const int k0 = inter ? s * 32 : (s - steps_d) * 32;
    for (int i = tid; i < 32 * CH; i += 256) {
      const int r = i >> 5, x = i & 31;
      if (SSD) {
        float a = 0.f;
        if (inter) {
          if (r < cd.y && k0 + x < D) a = crow[(size_t)r * CD + k0 + x] * eg[r];
        } else if (k0 + x <= r && r < cd.y) {
          const float2 gi = gs[r], gj = gs[k0 + x];
          a = cb[r * CH + k0 + x] * dts[k0 + x] * expf((gi.x - gj.x) + (gi.y - gj.y));
        }
        As[x][r] = a;
      } else if (inter) As[x][r] = k0 + x < D ? wk.qt[(ch * CH + r) * D + k0 + x] : 0.f;
      else As[x][r] = wk.P[(ch * CH + r) * CH + k0 + x];
    }
    for (int i = tid; i < 32 * 64; i += 256) {
      const int x = i >> 6, v = i & 63;
      float b = 0.f;
      if (v0 + v < V) {
        if (inter) b = k0 + x < D ? wk.KV[(ch * D + k0 + x) * V + v0 + v] : 0.f;
        else if (SSD) b = k0 + x < cd.y ? xrow[(size_t)(k0 + x) * CD + h * V + v0 + v] : 0.f;
        else b = k0 + x < cd.y ? mx.proj[(size_t)(cd.x + k0 + x) * mx.ld + mx.ov + h * V + v0 + v] : 0.f;
      }
      Bs[x][v] = b;
    }
    __syncthreads();
#pragma unroll 8
    for (int x = 0; x < 32; ++x) {
      const float4 a = *reinterpret_cast<const float4*>(&As[x][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&Bs[x][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    if (want_n) {
      for (int x = 0; x < 32; ++x) {
        if (inter) nq = k0 + x < D ? fmaf(As[x][tid], wk.NK[ch * D + k0 + x], nq) : nq;
        else nq += As[x][tid];
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= cd.y) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int v = v0 + tx * 4 + j;
      if (SSD && v < V) acc[i][j] = fmaf(mx.skip[h], xrow[(size_t)r * CD + h * V + v], acc[i][j]);
      if (v < V) raw.o[((size_t)(cd.x + r) * mx.H + h) * V + v] = acc[i][j];
    }
  }
  if (want_n && tid < cd.y) raw.nq[(size_t)(cd.x + tid) * mx.H + h] = nq;
}

// ---------------------------------------------------------------------------------------
// normalisation, output gate

// One block per (head, row). norm_w: [H * V] (per_head = 0), [V] shared by the heads, or null (no weight). last_slot[row] = slot whose portion
// ends at this row, or -1: mLSTM's running maximum is stored there once every reader of the old one is done.
template <int KIND, typename OutT>
__global__ void __launch_bounds__(256) state_out_kernel(const Mixer mx, const Raw raw, const float* norm_w, int per_head, float eps,
                                                        const int* last_slot, OutT* out, int ldo) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  constexpr int KEEP = 4;       // values per thread that stay in registers between the two passes
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, nt = blockDim.x;
  const int H = mx.H, V = mx.V;
  const size_t unit = (size_t)t * H + h;
  const float* o = raw.o + unit * V;
  const float* gate = mx.proj + (size_t)t * mx.ld + mx.og + h * V;
  float x[KEEP], z[KEEP], inv = 1.f, ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = tid + i * nt;
    x[i] = v < V ? o[v] : 0.f;
    z[i] = KIND != KIND_HGRN && v < V ? gate[v] : 0.f;
  }
  if (KIND == KIND_MLSTM) {
    const float m = raw.m[unit];
    inv = 1.f / (fmaxf(fabsf(raw.nq[unit]), expf(-m)) + 1e-6f);
    if (tid == 0 && last_slot[t] >= 0) mx.Ms[(size_t)last_slot[t] * H + h] = m;
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i) ss = fmaf(x[i] * inv, x[i] * inv, ss);
  for (int v = tid + KEEP * nt; v < V; v += nt) ss = fmaf(o[v] * inv, o[v] * inv, ss);
  const float r = inv / sqrtf(block_sum(ss, scratch) / (float)V + eps);
  OutT* dst = out + (size_t)t * ldo + h * V;
  const float* w = norm_w ? norm_w + (per_head ? 0 : h * V) : nullptr;
  auto put = [&](int v, float xv, float zv) {
    const float s = 1.f / (1.f + expf(-zv));
    dst[v] = (OutT)(xv * r * (w ? w[v] : 1.f) * (KIND == KIND_HGRN ? 1.f : KIND == KIND_MLSTM ? s : zv * s));
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if (tid + i * nt < V) put(tid + i * nt, x[i], z[i]);
  for (int v = tid + KEEP * nt; v < V; v += nt) put(v, o[v], KIND != KIND_HGRN ? gate[v] : 0.f);
  if (h == H - 1)
    for (int v = H * V + tid; v < ldo; v += nt) out[(size_t)t * ldo + v] = (OutT)0.f;
}

template <int KIND>
int launch_rows(const Mixer& mx, const Raw& raw, const int4* seqs, int nseq, cudaStream_t stream) {
  const int cols = mx.V + (KIND == KIND_MLSTM ? 1 : 0);
  const dim3 grid((cols + 31) / 32, mx.H, nseq);
  const size_t smem = (size_t)(3 * mx.D + GR * 33) * sizeof(float);
  const int rpt = (mx.D + GR - 1) / GR;
#define PK_ROWS_CASE(n)                                                                             \
  if (rpt <= n) {                                                                                   \
    PK_LAUNCH_PDL((state_rows_kernel<KIND, n>), grid, dim3(32 * GR), smem, stream, mx, raw, seqs);  \
    return PK_OK;                                                                                   \
  }
  PK_ROWS_CASE(4)
  PK_ROWS_CASE(8)
  PK_ROWS_CASE(16)
  PK_ROWS_CASE(32)
  PK_ROWS_CASE(64)
#undef PK_ROWS_CASE
  return PK_ERR_UNSUPPORTED;
}

size_t align4(size_t n) { return (n + 3) & ~(size_t)3; }

Work carve(float* ws, const Mixer& mx, int nchunks, int kind, size_t* total) {
  const size_t c = (size_t)nchunks, H = mx.H, D = mx.D, V = mx.V;
  size_t off = 0;
  Work w{};
  auto take = [&](size_t n) {
    float* p = ws ? ws + off : nullptr;
    off += align4(n);
    return p;
  };
  if (kind == KIND_GLA) w.logd = take(c * CH * H * D);
  if (kind == KIND_MLSTM) {
    w.lf = take(c * CH * H);
    w.ig = take(c * CH * H);
    w.NK = take(c * H * D);
  }
  w.dec_w = kind == KIND_SSD ? 1 : mx.D;
  w.dec = take(c * H * w.dec_w);
  if (kind == KIND_SSD) {
    w.xbc = take(c * CH * ssd_channels(mx));
    w.dt = take(c * H * CH);
    w.G = (float2*)take(c * H * CH * 2);
    w.P = take(c * mx.groups * CH * CH);
  } else {
    w.qt = take(c * H * CH * D);
    w.kt = take(c * H * CH * D);
    w.P = take(c * H * CH * CH);
  }
  w.KV = take(c * H * D * V);
  *total = off;
  return w;
}

}  // namespace

static bool unpack(const PkStateMixer* d, Mixer& mx, Raw& raw) {
  if (d == nullptr || d->proj == nullptr || d->S == nullptr || d->o == nullptr || d->H < 1 || d->D < 1 || d->V < 1 || d->D > 512) return false;
  if (d->kind == KIND_MLSTM && (!d->bi || !d->bf || !d->N || !d->Ms || !d->nq || !d->m || !(d->cap > 0.f))) return false;
  if (d->kind == KIND_GLA && (!d->a2 || !d->a2b || d->rank < 1 || d->rank > 1024)) return false;
  if (d->kind == KIND_RETENTION && (!d->pw || d->rot < 0 || (d->rot & 1) != 0 || d->rot > d->D || (d->rot > 0 && !d->freq))) return false;
  if (d->kind == KIND_SSD && (!d->cw || !d->cb || !d->dtb || !d->A || !d->skip || d->groups < 1 || d->H % d->groups != 0 || d->taps < 1 ||
                              (d->taps > 1 && !d->Cs)))
    return false;
  if (d->kind == KIND_HGRN && (!d->bf || !d->low)) return false;
  if (d->kind < KIND_GLA || d->kind > KIND_HGRN) return false;
  mx = Mixer{d->proj, d->ld, d->oq, d->ok, d->ov, d->og, d->oi, d->of, d->oa, d->H, d->D, d->V, d->qscale, d->bi, d->bf,
             d->cap, d->a2, d->a2b, d->rank, d->inv_tau, d->freq, d->rot, d->pw, d->cw, d->cb, d->dtb, d->A, d->skip, d->Cs,
             d->groups, d->taps, d->odt, d->low, d->S, d->N, d->Ms};
  raw = Raw{d->o, d->nq, d->m};
  return true;
}

// Tokens of short portions, one after the other. seqs [nseq] = {first row, tokens, slot, first position}.
PK_API int pk_state_rows(const PkStateMixer* d, const void* seqs, int nseq, cudaStream_t stream) {
  Mixer mx;
  Raw raw;
  if (!unpack(d, mx, raw) || seqs == nullptr || nseq < 1) return PK_ERR_BAD_ARG;
  switch (d->kind) {
    case KIND_GLA: return launch_rows<KIND_GLA>(mx, raw, (const int4*)seqs, nseq, stream);
    case KIND_SSD: return PK_ERR_UNSUPPORTED;      // pk_ssd_rows
    case KIND_MLSTM: return launch_rows<KIND_MLSTM>(mx, raw, (const int4*)seqs, nseq, stream);
    case KIND_HGRN: return launch_rows<KIND_HGRN>(mx, raw, (const int4*)seqs, nseq, stream);
    default: return launch_rows<KIND_RETENTION>(mx, raw, (const int4*)seqs, nseq, stream);
  }
}

// Workspace floats of pk_state_chunks.
PK_API size_t pk_state_chunk_workspace(const PkStateMixer* d, int nchunks) {
  Mixer mx{};
  mx.H = d->H;
  mx.D = d->D;
  mx.V = d->V;
  mx.groups = d->groups;
  size_t n = 0;
  carve(nullptr, mx, nchunks, d->kind, &n);
  return n;
}

// Long portions in chunks of 64. seqs [nseq] as above, chunks [nchunks] = {first row, tokens (1..64), sequence, chunk of the
// sequence}, chunk0 [nseq] = first chunk of each sequence (its chunks are consecutive).
PK_API int pk_state_chunks(const PkStateMixer* d, const void* seqs, int nseq, const void* chunks, const int* chunk0, int nchunks,
                           float* ws, cudaStream_t stream) {
  Mixer mx;
  Raw raw;
  if (!unpack(d, mx, raw) || seqs == nullptr || chunks == nullptr || chunk0 == nullptr || nseq < 1 || nchunks < nseq || ws == nullptr ||
      ((uintptr_t)ws & 15) != 0)
    return PK_ERR_BAD_ARG;
  size_t n = 0;
  const Work wk = carve(ws, mx, nchunks, d->kind, &n);
  const Chunks ck{(const int4*)seqs, (const int4*)chunks, chunk0, nseq, nchunks};
  const int H = mx.H, dt = (mx.D + 63) / 64, vt = (mx.V + 63) / 64;
  if (d->kind == KIND_GLA) {
    const int z = (H * mx.D + 255) / 256;
    gla_gates_kernel<<<dim3(nchunks, CH / 8, z < 16 ? z : 16), 256, (size_t)8 * mx.rank * sizeof(float), stream>>>(mx, ck, wk);
    PK_CHECK_LAUNCH();
    gla_intra_kernel<KIND_GLA><<<dim3(nchunks, H), 256, 0, stream>>>(mx, ck, wk);
  } else if (d->kind == KIND_HGRN) {
    gla_intra_kernel<KIND_HGRN><<<dim3(nchunks, H), 256, 0, stream>>>(mx, ck, wk);
  } else if (d->kind == KIND_SSD) {
    const int cb = (ssd_channels(mx) + 255) / 256;
    const dim3 grid(nchunks, cb + (H + 7) / 8);
    if (mx.taps == 2) ssd_inputs_kernel<2><<<grid, 256, 0, stream>>>(mx, ck, wk, cb);
    else if (mx.taps == 3) ssd_inputs_kernel<3><<<grid, 256, 0, stream>>>(mx, ck, wk, cb);
    else if (mx.taps == 4) ssd_inputs_kernel<4><<<grid, 256, 0, stream>>>(mx, ck, wk, cb);
    else ssd_inputs_kernel<0><<<grid, 256, 0, stream>>>(mx, ck, wk, cb);
    PK_CHECK_LAUNCH();
    ssd_scores_kernel<<<dim3(nchunks, mx.groups), 256, 0, stream>>>(mx, ck, wk);
  } else if (d->kind == KIND_RETENTION) {
    retention_intra_kernel<<<dim3(nchunks, H), 256, 0, stream>>>(mx, ck, wk);
  } else {
    mlstm_gates_kernel<<<dim3(nseq, H), 256, 0, stream>>>(mx, raw, ck, wk);
    PK_CHECK_LAUNCH();
    mlstm_intra_kernel<<<dim3(nchunks, H), 256, 0, stream>>>(mx, raw, ck, wk);
  }
  PK_CHECK_LAUNCH();
  const bool ssd = d->kind == KIND_SSD;
  if (ssd) chunk_kv_kernel<true><<<dim3(nchunks, H, dt * vt), 256, 0, stream>>>(mx, ck, wk, dt);
  else chunk_kv_kernel<false><<<dim3(nchunks, H, dt * vt), 256, 0, stream>>>(mx, ck, wk, dt);
  PK_CHECK_LAUNCH();
  const bool v4 = (mx.V & 3) == 0 && ((uintptr_t)mx.S & 15) == 0;
  const int elems = mx.D * mx.V / (v4 ? 4 : 1) + (d->kind == KIND_MLSTM ? mx.D : 0);
  const dim3 scan_grid((elems + 255) / 256, H, nseq);
  if (v4) chunk_scan_kernel<4><<<scan_grid, 256, 0, stream>>>(mx, ck, wk);
  else chunk_scan_kernel<1><<<scan_grid, 256, 0, stream>>>(mx, ck, wk);
  PK_CHECK_LAUNCH();
  if (ssd) chunk_out_kernel<true><<<dim3(nchunks, H, vt), 256, 0, stream>>>(mx, raw, ck, wk);
  else chunk_out_kernel<false><<<dim3(nchunks, H, vt), 256, 0, stream>>>(mx, raw, ck, wk);
  PK_CHECK_LAUNCH();
  return PK_OK;
}

// Head norm, output gate (SiLU; mLSTM: sigmoid; HGRN2: none) and running-maximum write-back for all rows of a step. norm_w null: no weight.
PK_API int pk_state_out(const PkStateMixer* d, const float* norm_w, int per_head, float eps, const int* last_slot, int rows, void* out,
                        int ldo, int out_f32, cudaStream_t stream) {
  Mixer mx;
  Raw raw;
  if (!unpack(d, mx, raw) || last_slot == nullptr || rows < 1 || out == nullptr || ldo < mx.H * mx.V) return PK_ERR_BAD_ARG;
  if (rows > 65535) return PK_ERR_BAD_ARG;
  const int nt = (mx.V + 31) / 32 * 32;
  const dim3 grid(mx.H, rows), block(nt < 256 ? nt : 256);
#define PK_OUT_CASE(kind)                                                                                                                                     \
  if (out_f32) PK_LAUNCH_PDL((state_out_kernel<kind, float>), grid, block, (size_t)0, stream, mx, raw, norm_w, per_head, eps, last_slot, (float*)out, ldo);   \
  else PK_LAUNCH_PDL((state_out_kernel<kind, pk::bf16>), grid, block, (size_t)0, stream, mx, raw, norm_w, per_head, eps, last_slot, (pk::bf16*)out, ldo)
  if (d->kind == KIND_MLSTM) PK_OUT_CASE(KIND_MLSTM);
  else if (d->kind == KIND_HGRN) PK_OUT_CASE(KIND_HGRN);
  else PK_OUT_CASE(KIND_GLA);
#undef PK_OUT_CASE
  return PK_OK;
}
