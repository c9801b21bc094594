// State-space recurrence of Mamba-2 (linear_state.cu has its equations and the fp32 chunk form).
//
// Rows form (decode, portions of a few tokens): one block per (sequence, head, 32 or 64 value columns), the state slice in
// registers, tokens in order; the convolution is part of it. A last kernel gates and norms the outputs of all rows and keeps
// the inputs that later convolutions need.
//
// Tiles (long portions of bf16 models) on the 5th-generation tensor cores: the chunked form over 128 tokens,
//   y_i = e^{G_i} C_i S_c + sum_{j <= i} (C_i . B_j) e^{G_i - G_j} dt_j x_j + D x_i,     S_{c+1} = e^{G_end} S_c + sum_j B_j (dt_j e^{G_end - G_j} x_j)^T
// with G the running log decay. x, B and C behind their convolution are bf16; what the recurrence makes of them is not: the
// state, the factors and the sums are fp32, and a fp32 operand enters a product as the sum of two bf16 terms (16 significant
// bits).
//
//   inputs  convolution and SiLU into rows of [x heads, VP each | B groups, 128 each | C groups, 128 each] (bf16, zero padded, rows
//           behind a tile's last token zero), step sizes and running log decays
//   kv      one CTA per (tile, head): sum_j B_j (w_j x_j)^T, both operands MN-major (their rows are tokens)
//   scan    over the tiles of a portion: the state before every tile, and the one behind the last
//   out     one CTA per (tile, head): S = C B^T and O = C S_c from TMA'd C and B; S times its factors goes back to shared memory,
//           over B and S_c which are done with, and is multiplied with x
// TMA loads have no multicast. Every wait is bounded (status word + CTA-wide abort flag).
#include "../common/pk_sm100.cuh"
#include "../common/pk_state.cuh"
#include "../common/pk_vec.cuh"

namespace {

using namespace pk;
using namespace pk::sm100;

// ---------------------------------------------------------------------------------------
// rows

constexpr int GR = 8;   // row groups (warps) of a block

template <int RPT, int TAPS, int VW>      // state rows per thread, taps (0: any number), adjacent value columns per thread
__global__ void __launch_bounds__(32 * GR) ssd_rows_kernel(const PkStateMixer m, const int4* seqs) {
  pdl_trigger();
  pdl_wait();
  constexpr int W = 32 * VW;
  extern __shared__ float sm[];
  float* qs = sm;                 // [D] C
  float* ks = qs + m.D;           // [D] B
  float* xs = ks + m.D;           // [W] x
  float* red = xs + W;            // [GR][W]
  __shared__ float s_sc[2];
  const int4 sq = seqs[blockIdx.z];          // first row, tokens, slot, first position
  const int h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, g = tid >> 5;
  const int D = m.D, V = m.V, col0 = blockIdx.x * W, col = col0 + lane * VW;
  const bool live = col < V;                 // VW 2: V is even
  float* Sp = m.S + ((size_t)sq.z * m.H + h) * D * V + col;
  float s[RPT][VW];
#pragma unroll
  for (int j = 0; j < RPT; ++j) {
    const int d = g + j * GR;
#pragma unroll
    for (int k = 0; k < VW; ++k) s[j][k] = 0.f;
    if (live && d < D && sq.w > 0) {
      if (VW == 2) {
        const float2 v = *reinterpret_cast<const float2*>(Sp + (size_t)d * V);
        s[j][0] = v.x;
        s[j][1 % VW] = v.y;
      } else {
        s[j][0] = Sp[(size_t)d * V];
      }
    }
  }
  const int b0 = m.H * V + h / (m.H / m.groups) * D;
  const float skip = m.skip[h];
  for (int t = 0; t < sq.y; ++t) {
    const int row = sq.x + t, pos = sq.w + t;
    for (int i = tid; i < 2 * D; i += 32 * GR) {
      const bool is_q = i >= D;
      const int d = is_q ? i - D : i;
      (is_q ? qs : ks)[d] = conv_silu<TAPS>(m, sq.z, row, t, pos, b0 + (is_q ? m.groups * D : 0) + d);
    }
    if (tid < W && col0 + tid < V) xs[tid] = conv_silu<TAPS>(m, sq.z, row, t, pos, h * V + col0 + tid);
    if (tid == 32 * GR - 1) {
      const float dt = softplus(m.proj[(size_t)row * m.ld + m.odt + h] + m.dtb[h]);
      s_sc[0] = expf(m.A[h] * dt);
      s_sc[1] = dt;
    }
    __syncthreads();
    float v[VW], part[VW];
#pragma unroll
    for (int k = 0; k < VW; ++k) {
      v[k] = live ? xs[lane * VW + k] * s_sc[1] : 0.f;
      part[k] = 0.f;
    }
    const float a = s_sc[0];
#pragma unroll
    for (int j = 0; j < RPT; ++j) {
      const int d = g + j * GR;
      if (d < D) {
        const float kd = ks[d], qd = qs[d];
#pragma unroll
        for (int k = 0; k < VW; ++k) {
          s[j][k] = fmaf(a, s[j][k], kd * v[k]);
          part[k] = fmaf(s[j][k], qd, part[k]);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < VW; ++k) red[g * W + lane * VW + k] = part[k];
    __syncthreads();
    if (tid < W && col0 + tid < V) {
      float o = skip * xs[tid];
#pragma unroll
      for (int i = 0; i < GR; ++i) o += red[i * W + tid];
      m.o[((size_t)row * m.H + h) * V + col0 + tid] = o;
    }
    if (t + 1 < sq.y) __syncthreads();
  }
  if (live) {
#pragma unroll
    for (int j = 0; j < RPT; ++j) {
      const int d = g + j * GR;
      if (d < D) {
        if (VW == 2) *reinterpret_cast<float2*>(Sp + (size_t)d * V) = make_float2(s[j][0], s[j][1 % VW]);
        else Sp[(size_t)d * V] = s[j][0];
      }
    }
  }
}

template <int TAPS, int VW>
int launch_rows(const PkStateMixer& m, const int4* seqs, int nseq, cudaStream_t stream) {
  const dim3 grid((m.V + 32 * VW - 1) / (32 * VW), m.H, nseq);
  const size_t smem = (size_t)(2 * m.D + (GR + 1) * 32 * VW) * sizeof(float);
  const int rpt = (m.D + GR - 1) / GR;
#define PK_ROWS_CASE(n)                                                                           \
  if (rpt <= n) {                                                                                 \
    PK_LAUNCH_PDL((ssd_rows_kernel<n, TAPS, VW>), grid, dim3(32 * GR), smem, stream, m, seqs);    \
    return PK_OK;                                                                                 \
  }
  PK_ROWS_CASE(4)
  PK_ROWS_CASE(8)
  PK_ROWS_CASE(16)
  PK_ROWS_CASE(32)
  PK_ROWS_CASE(64)
#undef PK_ROWS_CASE
  return PK_ERR_UNSUPPORTED;
}

template <int VW>
int launch_rows(const PkStateMixer& m, const int4* seqs, int nseq, cudaStream_t stream) {
  if (m.taps == 4) return launch_rows<4, VW>(m, seqs, nseq, stream);
  if (m.taps == 3) return launch_rows<3, VW>(m, seqs, nseq, stream);
  return launch_rows<0, VW>(m, seqs, nseq, stream);
}

// ---------------------------------------------------------------------------------------
// gate, norm

// y silu(z), normed in gridDim.x equal parts of the heads' outputs laid end to end, times norm_w [H * V]. One block per (part,
// row); columns from H * V up to `width` are set to zero. behind[row]: tokens of the same portion after the row; the last rows of
// a portion leave their inputs in the convolution's ring.
template <typename OutT, int VW>
__global__ void __launch_bounds__(1024) ssd_out_kernel(const PkStateMixer m, const float* norm_w, float eps, const int* slots, const int* behind, const int* pos,
                                                       OutT* out, int ldo, int width) {
  pdl_trigger();
  pdl_wait();
  __shared__ float scratch[33];
  constexpr int KEEP = 4;
  const int g = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, nt = blockDim.x;
  const int inner = m.H * m.V, n = inner / gridDim.x;
  if (behind[t] < m.taps - 1) {
    const int CD = ssd_channels(m), step = gridDim.x * nt;
    const float* src = m.proj + (size_t)t * m.ld + m.ov;
    float* ring = m.Cs + ((size_t)slots[t] * (m.taps - 1) + pos[t] % (m.taps - 1)) * CD;
    for (int ch = g * nt + tid; ch < CD; ch += 4 * step) {
      float in[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) in[i] = ch + i * step < CD ? src[ch + i * step] : 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (ch + i * step < CD) ring[ch + i * step] = in[i];
    }
  }
  const float* o = m.o + (size_t)t * inner + g * n;
  const float* gate = m.proj + (size_t)t * m.ld + m.og + g * n;
  auto gated = [&](int v, float (&x)[VW]) {
    float z[VW];
    load_f32<VW>(o + v, x);
    load_f32<VW>(gate + v, z);
#pragma unroll
    for (int k = 0; k < VW; ++k) x[k] *= silu_exact(z[k]);
  };
  float x[KEEP][VW], ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = (tid + i * nt) * VW;
    if (v >= n) continue;
    gated(v, x[i]);
#pragma unroll
    for (int k = 0; k < VW; ++k) ss = fmaf(x[i][k], x[i][k], ss);
  }
  for (int v = (tid + KEEP * nt) * VW; v < n; v += nt * VW) {
    float y[VW];
    gated(v, y);
#pragma unroll
    for (int k = 0; k < VW; ++k) ss = fmaf(y[k], y[k], ss);
  }
  const float r = 1.f / sqrtf(block_sum(ss, scratch) / (float)n + eps);
  OutT* dst = out + (size_t)t * ldo + g * n;
  auto put = [&](int v, float (&y)[VW]) {
    float w[VW];
    load_f32<VW>(norm_w + g * n + v, w);
#pragma unroll
    for (int k = 0; k < VW; ++k) y[k] *= r * w[k];
    store<VW>(dst + v, y);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if ((tid + i * nt) * VW < n) put((tid + i * nt) * VW, x[i]);
  for (int v = (tid + KEEP * nt) * VW; v < n; v += nt * VW) {
    float y[VW];
    gated(v, y);
    put(v, y);
  }
  if (g == gridDim.x - 1)
    for (int v = inner + tid; v < width; v += nt) out[(size_t)t * ldo + v] = (OutT)0.f;
}

template <typename OutT, int VW>
int launch_out(const PkStateMixer& m, const float* norm_w, int parts, float eps, const int* slots, const int* behind, const int* pos, int rows, OutT* out, int ldo,
               int width, cudaStream_t stream) {
  const int groups = (m.H * m.V / parts + VW - 1) / VW, per = rows > 64 ? 2 : 1;
  int nt = ((groups + per - 1) / per + 31) / 32 * 32;
  if (nt > 1024) nt = 1024;
  PK_LAUNCH_PDL((ssd_out_kernel<OutT, VW>), dim3(parts, rows), dim3(nt), (size_t)0, stream, m, norm_w, eps, slots, behind, pos, out, ldo, width);
  return PK_OK;
}

// ---------------------------------------------------------------------------------------
// tiles

constexpr int L = 128;               // tokens of a tile
constexpr int NP = 128;              // padded state dimension
constexpr int kPanel = L * 128;      // bytes of 128 rows of 64 bf16

struct Params {
  PkStateMixer m;
  const int4* tiles;       // {first step row, rows, portion, unused}
  const int4* seqs;        // {first step row, tokens, slot, first position}
  const int* tile0;        // first tile of every portion
  bf16* xbc;               // [tiles x 128, cols]
  float* dt;               // [tile, H, 128]
  float2* G;               // [tile, H, 128]
  float* dec;              // [tile, H]
  float* KV;               // [tile, H, D, V] sums of a tile, then the state before it
  int cols, vp;
  uint32_t* status;
};

template <int TAPS>
__global__ void __launch_bounds__(256) ssd_tile_inputs_kernel(const Params p, int conv_blocks) {
  const PkStateMixer& m = p.m;
  const int c = blockIdx.x, tid = threadIdx.x;
  const int4 cd = p.tiles[c], sq = p.seqs[cd.z];
  if ((int)blockIdx.y >= conv_blocks) {
    const int h = (blockIdx.y - conv_blocks) * 8 + (tid >> 5), lane = tid & 31;
    if (h >= m.H || blockIdx.z > 0) return;
    const size_t at = (size_t)c * m.H + h;
    float total;
    ssd_decays<L / 32>(m, cd.x, cd.y, h, lane, p.dt + at * L, p.G + at * L, &total);
    if (lane == 31) p.dec[at] = expf(total);
    return;
  }
  const int col = blockIdx.y * 256 + tid;
  if (col >= p.cols) return;
  // channel of this column, -1: padding
  const int xw = m.H * p.vp;
  int ch = -1;
  if (col < xw) {
    const int h = col / p.vp, v = col - h * p.vp;
    if (v < m.V) ch = h * m.V + v;
  } else {
    const int g = (col - xw) / NP, n = (col - xw) % NP;
    if (n < m.D) ch = m.H * m.V + g * m.D + n;      // B groups, then C groups
  }
  const int rows = L / gridDim.z, r0 = blockIdx.z * rows, n = ch < 0 ? 0 : min(max(cd.y - r0, 0), rows);
  const int t0 = cd.x - sq.x + r0;
  bf16* out = p.xbc + ((size_t)c * L + r0) * p.cols + col;
  if (n > 0) conv_silu_rows<TAPS>(m, sq.z, cd.x + r0, t0, sq.w + t0, n, ch, [&](int r, float y) { out[(size_t)r * p.cols] = __float2bfloat16(y); });
  for (int r = n; r < rows; ++r) out[(size_t)r * p.cols] = __float2bfloat16(0.f);
}

__device__ __forceinline__ uint64_t desc_mn_sw128(uint32_t smem_addr, uint32_t panel) {      // see attention_prefill.cu
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3ffffu) >> 4);
  d |= (uint64_t)((panel >> 4) & 0x3fffu) << 16;
  d |= (uint64_t)((1024u >> 4) & 0x3fffu) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

// Two fp32 as the packed leading bf16 terms, and the packed remainders.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const bf162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const bf162 l = __floats2bfloat162_rn(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xffff0000u));
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

__device__ __forceinline__ void unpack8(const uint4& u, float (&f)[8]) {
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(w[i] << 16);
    f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
  }
}

struct Ctl {
  uint64_t load, x_full, done1, done2;
  uint32_t tmem_base;
  volatile uint32_t abort_flag;
};

// rows 0 .. 127 of one panel (64 columns from x on)
__device__ __forceinline__ void load_panel(uint8_t* dst, const CUtensorMap* map, uint64_t* bar, int x, int y) {
  tma_load_2d(dst, map, bar, x, y);
  tma_load_2d(dst + kPanel / 2, map, bar, x, y + L / 2);
}

// All threads see the tensor memory's address and initialised barriers behind this.
__device__ __forceinline__ void setup(Ctl& ct, int warp, uint32_t cols) {
  if (threadIdx.x == 0) {
    mbar_init(&ct.load, 1);
    mbar_init(&ct.x_full, 1);
    mbar_init(&ct.done1, 1);
    mbar_init(&ct.done2, 1);
    ct.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(&ct.tmem_base, cols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
}

__device__ __forceinline__ void drain(uint64_t* bar) {
  for (uint32_t i = 0; i < (1u << 20); ++i)
    if (mbar_try_wait(bar, 0)) break;
}

template <int VP>
__global__ void __launch_bounds__(128) ssd_tile_kv_kernel(const __grid_constant__ CUtensorMap tmap, const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int NV = VP / 64;
  uint8_t* sb = base;                       // B: two panels
  uint8_t* sx = sb + 2 * kPanel;            // w x: [2 terms][NV] panels
  Ctl& ct = *reinterpret_cast<Ctl*>(sx + 2 * NV * kPanel);
  const PkStateMixer& m = p.m;
  const int h = blockIdx.x, c = blockIdx.y, tid = threadIdx.x, warp = tid >> 5;
  const size_t unit = (size_t)c * m.H + h;
  setup(ct, warp, VP);
  const uint32_t acc = ct.tmem_base;
  if (tid == 0) {
    const int x = m.H * VP + h / (m.H / m.groups) * NP;
    mbar_arrive_expect_tx(&ct.load, 2 * kPanel);
    load_panel(sb, &tmap, &ct.load, x, c * L);
    load_panel(sb + kPanel, &tmap, &ct.load, x + 64, c * L);
  }
  {
    const float2 g = p.G[unit * L + tid], e = p.G[unit * L + L - 1];
    const float w = p.dt[unit * L + tid] * expf((e.x - g.x) + (e.y - g.y));
    const uint4* src = reinterpret_cast<const uint4*>(p.xbc + ((size_t)c * L + tid) * p.cols + h * VP);
    uint4 raw[VP / 8];
#pragma unroll
    for (int k = 0; k < VP / 8; ++k) raw[k] = src[k];
#pragma unroll
    for (int k = 0; k < VP / 8; ++k) {
      float f[8];
      unpack8(raw[k], f);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) split2(f[2 * i] * w, f[2 * i + 1] * w, hi[i], lo[i]);
      uint8_t* dst = sx + (k >> 3) * kPanel + tid * 128 + (((k & 7) ^ (tid & 7)) << 4);
      *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(dst + NV * kPanel) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 0) {
    if (mbar_wait(&ct.load, 0, &ct.abort_flag, p.status, 80)) {
      constexpr uint32_t idesc = umma_idesc(1, 1, L, VP) | (1u << 15) | (1u << 16);      // both MN-major
      const uint32_t a = smem_u32(sb), b = smem_u32(sx);
#pragma unroll
      for (int j = 0; j < 16; ++j)      // eight steps of 16 tokens with the leading terms, then with the remainders
        umma_f16(acc, desc_mn_sw128(a + (j & 7) * 2048, kPanel), desc_mn_sw128(b + (j >> 3) * NV * kPanel + (j & 7) * 2048, kPanel), idesc, j > 0 ? 1u : 0u);
      umma_commit(&ct.done1);
    } else {
      drain(&ct.load);
    }
  }
  if (mbar_wait_warp(&ct.done1, 0, &ct.abort_flag, p.status, 81)) {
    tc_fence_after();
    const int n = tid;
    float* dst = p.KV + (unit * m.D + n) * m.V;
#pragma unroll 1
    for (int k = 0; k < VP / 32; ++k) {
      uint32_t r[32];
      tmem_ld_32x32(acc + ((uint32_t)(warp * 32) << 16) + k * 32, r);
      tmem_ld_wait();
      if (n >= m.D) continue;
      if ((m.V & 3) == 0) {
#pragma unroll
        for (int i = 0; i < 32; i += 4)
          if (k * 32 + i < m.V) *reinterpret_cast<uint4*>(dst + k * 32 + i) = make_uint4(r[i], r[i + 1], r[i + 2], r[i + 3]);
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (k * 32 + i < m.V) dst[k * 32 + i] = __uint_as_float(r[i]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(ct.tmem_base, VP);
  }
}

// Serial over a portion's tiles, one thread per VW adjacent state elements.
template <int VW>
__global__ void __launch_bounds__(256) ssd_tile_scan_kernel(const Params p) {
  const PkStateMixer& m = p.m;
  const int4 sq = p.seqs[blockIdx.z];
  const int h = blockIdx.y, e = (blockIdx.x * 256 + threadIdx.x) * VW;
  if (e >= m.D * m.V) return;
  const int c0 = p.tile0[blockIdx.z], n = (sq.y + L - 1) / L;
  float* state = m.S + ((size_t)sq.z * m.H + h) * m.D * m.V + e;
  float* kv = p.KV + ((size_t)c0 * m.H + h) * m.D * m.V + e;
  const float* dec = p.dec + (size_t)c0 * m.H + h;
  const size_t step = (size_t)m.H * m.D * m.V;
  constexpr int AHEAD = 8;
  float s[VW], add[AHEAD][VW], dc[AHEAD];
  auto load = [&](const float* q, float (&v)[VW]) {
    if (VW == 4) {
      const float4 x = *reinterpret_cast<const float4*>(q);
      v[0] = x.x; v[1 % VW] = x.y; v[2 % VW] = x.z; v[3 % VW] = x.w;
    } else {
      v[0] = *q;
    }
  };
  auto store = [&](float* q, const float (&v)[VW]) {
    if (VW == 4) *reinterpret_cast<float4*>(q) = make_float4(v[0], v[1 % VW], v[2 % VW], v[3 % VW]);
    else *q = v[0];
  };
#pragma unroll
  for (int i = 0; i < VW; ++i) s[i] = 0.f;
  if (sq.w > 0) load(state, s);
  for (int c = 0; c < n; c += AHEAD) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c + i < n) {
        load(kv + (size_t)(c + i) * step, add[i]);
        dc[i] = dec[(size_t)(c + i) * m.H];
      }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      if (c + i < n) {
        store(kv + (size_t)(c + i) * step, s);
#pragma unroll
        for (int k = 0; k < VW; ++k) s[k] = fmaf(dc[i], s[k], add[i][k]);
      }
  }
  store(state, s);
}

template <int VP>
__global__ void __launch_bounds__(128) ssd_tile_out_kernel(const __grid_constant__ CUtensorMap tmap, const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int NV = VP / 64;
  uint8_t* sc = base;                       // C: two panels; then x: NV panels
  uint8_t* sb = sc + 2 * kPanel;            // B: two panels
  uint8_t* ss = sb + 2 * kPanel;            // state: [2 terms][NV] panels. The weights, [2 terms][2] panels, lie over sb and ss
  Ctl& ct = *reinterpret_cast<Ctl*>(ss + 2 * NV * kPanel);
  float2* gs = reinterpret_cast<float2*>(&ct + 1);
  float* dts = reinterpret_cast<float*>(gs + L);
  const PkStateMixer& m = p.m;
  const int h = blockIdx.x, c = blockIdx.y, tid = threadIdx.x, warp = tid >> 5;
  const int4 tile = p.tiles[c];
  const size_t unit = (size_t)c * m.H + h;
  constexpr uint32_t kCols = 256;
  setup(ct, warp, kCols);
  const uint32_t t_s = ct.tmem_base, t_o = ct.tmem_base + L;      // S [128 columns], later S' x over it; C S_c
  if (tid == 0) {
    const int x = m.H * VP + h / (m.H / m.groups) * NP;
    mbar_arrive_expect_tx(&ct.load, 4 * kPanel);
    for (int i = 0; i < 2; ++i) {
      load_panel(sb + i * kPanel, &tmap, &ct.load, x + i * 64, c * L);
      load_panel(sc + i * kPanel, &tmap, &ct.load, x + m.groups * NP + i * 64, c * L);
    }
  }
  gs[tid] = p.G[unit * L + tid];
  dts[tid] = p.dt[unit * L + tid];
  {
    // state rows (one per state dimension) as two terms; 8 columns at a time, neighbouring threads on neighbouring pieces,
    // four pieces of a thread in flight
    const float* S = p.KV + unit * m.D * m.V;
    const bool v4 = (m.V & 3) == 0;
    constexpr int PIECES = VP / 8, AHEAD = 4;
#pragma unroll 1
    for (int i0 = tid; i0 < NP * PIECES; i0 += 128 * AHEAD) {
      float f[AHEAD][8];
#pragma unroll
      for (int a = 0; a < AHEAD; ++a) {
        const int n = (i0 + a * 128) / PIECES, k = (i0 + a * 128) % PIECES;
        const float* src = S + (size_t)n * m.V + k * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) f[a][e] = 0.f;
        if (n >= m.D) continue;
        if (v4) {
#pragma unroll
          for (int q = 0; q < 2; ++q)
            if (k * 8 + q * 4 < m.V) {
              const float4 x = *reinterpret_cast<const float4*>(src + q * 4);
              f[a][q * 4] = x.x; f[a][q * 4 + 1] = x.y; f[a][q * 4 + 2] = x.z; f[a][q * 4 + 3] = x.w;
            }
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (k * 8 + e < m.V) f[a][e] = src[e];
        }
      }
#pragma unroll
      for (int a = 0; a < AHEAD; ++a) {
        const int n = (i0 + a * 128) / PIECES, k = (i0 + a * 128) % PIECES;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split2(f[a][2 * e], f[a][2 * e + 1], hi[e], lo[e]);
        uint8_t* dst = ss + (k >> 3) * kPanel + n * 128 + (((k & 7) ^ (n & 7)) << 4);
        *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(dst + NV * kPanel) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
  }
  fence_proxy_async_smem();
  __syncthreads();
  const uint32_t ca = smem_u32(sc), ba = smem_u32(sb), sa = smem_u32(ss);
  constexpr uint32_t idesc_v = umma_idesc(1, 1, L, VP) | (1u << 16);       // second operand MN-major
  if (tid == 0) {
    if (mbar_wait(&ct.load, 0, &ct.abort_flag, p.status, 82)) {
      constexpr uint32_t idesc_s = umma_idesc(1, 1, L, L);
      const int steps = (m.D + 15) / 16;
      for (int j = 0; j < steps; ++j) {
        const uint64_t a = smem_desc_k_sw128(ca + (j >> 2) * kPanel + (j & 3) * 32);
        umma_f16(t_s, a, smem_desc_k_sw128(ba + (j >> 2) * kPanel + (j & 3) * 32), idesc_s, j > 0 ? 1u : 0u);
        umma_f16(t_o, a, desc_mn_sw128(sa + j * 2048, kPanel), idesc_v, j > 0 ? 1u : 0u);
        umma_f16(t_o, a, desc_mn_sw128(sa + NV * kPanel + j * 2048, kPanel), idesc_v, 1u);
      }
      umma_commit(&ct.done1);
    } else {
      drain(&ct.load);
    }
  }
  bool ok = mbar_wait_warp(&ct.done1, 0, &ct.abort_flag, p.status, 83);
  const uint32_t lane_off = (uint32_t)(warp * 32) << 16;
  bool x_issued = false;
  if (ok) {
    tc_fence_after();
    if (tid == 0) {      // the products above are done: x takes the place of C
      mbar_arrive_expect_tx(&ct.x_full, NV * kPanel);
      for (int i = 0; i < NV; ++i) load_panel(sc + i * kPanel, &tmap, &ct.x_full, h * VP + i * 64, c * L);
      x_issued = true;
    }
    const float2 gi = gs[tid];
#pragma unroll 1
    for (int k = 0; k < 4; ++k) {      // 32 columns; row of thread tid
      uint32_t r[32];
      if (k <= warp) {
        tmem_ld_32x32(t_s + lane_off + k * 32, r);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int j = k * 32 + i;
          const float2 gj = gs[j];
          const float f = j <= tid ? dts[j] * expf((gi.x - gj.x) + (gi.y - gj.y)) : 0.f;
          r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
        }
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i) r[i] = 0u;
      }
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) split2(__uint_as_float(r[q * 8 + 2 * e]), __uint_as_float(r[q * 8 + 2 * e + 1]), hi[e], lo[e]);
        uint8_t* dst = sb + (k >> 1) * kPanel + tid * 128 + ((((k & 1) * 4 + q) ^ (tid & 7)) << 4);
        *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(dst + 2 * kPanel) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
      }
    }
    fence_proxy_async_smem();
    tc_fence_before();
  }
  __syncthreads();
  if (tid == 0 && ok) {
    tc_fence_after();
    if (mbar_wait(&ct.x_full, 0, &ct.abort_flag, p.status, 84)) {
      const uint32_t wa = smem_u32(sb);
#pragma unroll
      for (int j = 0; j < 16; ++j)
        umma_f16(t_s, smem_desc_k_sw128(wa + (j >> 3) * 2 * kPanel + ((j & 7) >> 2) * kPanel + (j & 3) * 32), desc_mn_sw128(ca + (j & 7) * 2048, kPanel),
                 idesc_v, j > 0 ? 1u : 0u);
      umma_commit(&ct.done2);
    } else if (x_issued) {
      drain(&ct.x_full);
    }
  }
  if (ok && mbar_wait_warp(&ct.done2, 0, &ct.abort_flag, p.status, 85)) {
    tc_fence_after();
    mbar_wait(&ct.x_full, 0, &ct.abort_flag, p.status, 86);      // complete by now: every thread reads x below
    const float2 gi = gs[tid];
    const float eg = expf(gi.x + gi.y), sk = m.skip[h];
    float* dst = m.o + ((size_t)(tile.x + tid) * m.H + h) * m.V;
    const uint4* xs = reinterpret_cast<const uint4*>(sc);
#pragma unroll 1
    for (int k = 0; k < VP / 32; ++k) {
      uint32_t a[32], b[32];
      tmem_ld_32x32(t_s + lane_off + k * 32, a);
      tmem_ld_32x32(t_o + lane_off + k * 32, b);
      tmem_ld_wait();
      if (tid >= tile.y) continue;
      float y[32];
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        float x[8];
        unpack8(xs[((k >> 1) * kPanel + tid * 128 + ((((k & 1) * 4 + q) ^ (tid & 7)) << 4)) / 16], x);
#pragma unroll
        for (int e = 0; e < 8; ++e) y[q * 8 + e] = fmaf(sk, x[e], fmaf(eg, __uint_as_float(b[q * 8 + e]), __uint_as_float(a[q * 8 + e])));
      }
      if ((m.V & 3) == 0) {
#pragma unroll
        for (int i = 0; i < 32; i += 4)
          if (k * 32 + i < m.V) *reinterpret_cast<float4*>(dst + k * 32 + i) = make_float4(y[i], y[i + 1], y[i + 2], y[i + 3]);
      } else {
#pragma unroll
        for (int i = 0; i < 32; ++i)
          if (k * 32 + i < m.V) dst[k * 32 + i] = y[i];
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(ct.tmem_base, kCols);
  }
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*,
                                  const cuuint32_t*, const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle,
                                  CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiledFn encode_fn() {
  static EncodeTiledFn fn = nullptr;
  if (fn == nullptr) {
    void* sym = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &sym, cudaEnableDefault, &qres) == cudaSuccess && qres == cudaDriverEntryPointSuccess)
      fn = (EncodeTiledFn)sym;
  }
  return fn;
}

// `ws` floats, 256-byte aligned pieces
size_t carve(Params& p, float* ws, int ntiles) {
  const PkStateMixer& m = p.m;
  const size_t c = (size_t)ntiles, H = m.H;
  size_t off = 0;
  auto take = [&](size_t n) {
    float* q = ws ? ws + off : nullptr;
    off += (n + 63) & ~(size_t)63;
    return q;
  };
  p.vp = m.V <= 64 ? 64 : 128;
  p.cols = m.H * p.vp + 2 * m.groups * NP;
  p.xbc = (bf16*)take(c * L * p.cols / 2);
  p.dt = take(c * H * L);
  p.G = (float2*)take(c * H * L * 2);
  p.dec = take(c * H);
  p.KV = take(c * H * m.D * m.V);
  return off;
}

template <int VP>
int launch(const CUtensorMap& map, const Params& p, int ntiles, int nseq, cudaStream_t stream) {
  constexpr size_t ctl = sizeof(Ctl) + L * 12 + 16;
  constexpr size_t kv_smem = 1024 + (2 + 2 * (VP / 64)) * kPanel + sizeof(Ctl), out_smem = 1024 + (4 + 2 * (VP / 64)) * kPanel + ctl;
  static PkDeviceOnce once;
  if (PkDeviceOnceGuard g{once}; g.needed()) {
    if (cudaFuncSetAttribute(ssd_tile_kv_kernel<VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kv_smem) != cudaSuccess ||
        cudaFuncSetAttribute(ssd_tile_out_kernel<VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    g.done();
  }
  const PkStateMixer& m = p.m;
  const int cb = (p.cols + 255) / 256;
  const dim3 in_grid(ntiles, cb + (m.H + 7) / 8, 8);      // 16 rows per block
  if (m.taps == 2) ssd_tile_inputs_kernel<2><<<in_grid, 256, 0, stream>>>(p, cb);
  else if (m.taps == 3) ssd_tile_inputs_kernel<3><<<in_grid, 256, 0, stream>>>(p, cb);
  else if (m.taps == 4) ssd_tile_inputs_kernel<4><<<in_grid, 256, 0, stream>>>(p, cb);
  else ssd_tile_inputs_kernel<0><<<in_grid, 256, 0, stream>>>(p, cb);
  PK_CHECK_LAUNCH();
  ssd_tile_kv_kernel<VP><<<dim3(m.H, ntiles), 128, kv_smem, stream>>>(map, p);
  PK_CHECK_LAUNCH();
  const int e = m.D * m.V;
  if ((m.V & 3) == 0 && ((uintptr_t)m.S & 15) == 0) ssd_tile_scan_kernel<4><<<dim3((e / 4 + 255) / 256, m.H, nseq), 256, 0, stream>>>(p);
  else ssd_tile_scan_kernel<1><<<dim3((e + 255) / 256, m.H, nseq), 256, 0, stream>>>(p);
  PK_CHECK_LAUNCH();
  ssd_tile_out_kernel<VP><<<dim3(m.H, ntiles), 128, out_smem, stream>>>(map, p);
  PK_CHECK_LAUNCH();
  return PK_OK;
}

bool ssd_ok(const PkStateMixer* d) {
  return d != nullptr && d->proj != nullptr && d->S != nullptr && d->o != nullptr && d->cw != nullptr && d->cb != nullptr && d->dtb != nullptr && d->A != nullptr &&
         d->skip != nullptr && d->H >= 1 && d->D >= 1 && d->V >= 1 && d->groups >= 1 && d->H % d->groups == 0 && d->taps >= 1 && (d->taps == 1 || d->Cs != nullptr);
}

}  // namespace

// Workspace floats of pk_ssd_tiles; 0 when the shape does not fit it.
PK_API size_t pk_ssd_tile_workspace(const PkStateMixer* d, int ntiles) {
  if (d == nullptr || d->D > NP || d->V > 128) return 0;
  Params p{};
  p.m = *d;
  return carve(p, nullptr, ntiles);
}

// Outputs (in `o`) and states of long portions of a state-space layer. seqs [nseq] = {first row, tokens, slot, first position}, tiles
// [ntiles] = {first row, rows (1..128), portion, unused}, those of a portion one after the other from tile0[portion] on.
PK_API int pk_ssd_tiles(const PkStateMixer* d, const void* seqs, int nseq, const void* tiles, const int* tile0, int ntiles, float* ws, uint32_t* status,
                        cudaStream_t stream) {
  if (!ssd_ok(d) || seqs == nullptr || tiles == nullptr || tile0 == nullptr || nseq < 1 || ntiles < nseq || ntiles > 65535 || ws == nullptr || ((uintptr_t)ws & 255) != 0 ||
      ((uintptr_t)d->o & 15) != 0)
    return PK_ERR_BAD_ARG;
  if (d->D > NP || d->V > 128) return PK_ERR_UNSUPPORTED;
  EncodeTiledFn encode = encode_fn();
  if (encode == nullptr) return PK_ERR_UNSUPPORTED;
  Params p{};
  p.m = *d;
  p.seqs = (const int4*)seqs;
  p.tiles = (const int4*)tiles;
  p.tile0 = tile0;
  p.status = status;
  carve(p, ws, ntiles);
  CUtensorMap map;
  const cuuint64_t gdim[2] = {(cuuint64_t)p.cols, (cuuint64_t)ntiles * L}, gstride[1] = {(cuuint64_t)p.cols * 2};
  const cuuint32_t box[2] = {64, 64}, estr[2] = {1, 1};
  if (encode(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.xbc, gdim, gstride, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
             CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return PK_ERR_CUDA;
  return p.vp == 64 ? launch<64>(map, p, ntiles, nseq, stream) : launch<128>(map, p, ntiles, nseq, stream);
}

// Tokens of short portions, one after the other: outputs in `o`, states. seqs as above.
PK_API int pk_ssd_rows(const PkStateMixer* d, const void* seqs, int nseq, int sm_count, cudaStream_t stream) {
  if (!ssd_ok(d) || seqs == nullptr || nseq < 1 || d->D > 512) return PK_ERR_BAD_ARG;
  const long long blocks = (long long)((d->V + 31) / 32) * d->H * nseq;      // narrow ones, while the machine is not full
  if ((d->V & 1) == 0 && ((uintptr_t)d->S & 7) == 0 && blocks > 2LL * (sm_count > 0 ? sm_count : 148) && d->V > 32)
    return launch_rows<2>(*d, (const int4*)seqs, nseq, stream);
  return launch_rows<1>(*d, (const int4*)seqs, nseq, stream);
}

// Gate, norm in `parts` parts, output rows [rows, ldo] of which `width` columns are this layer's; the last inputs of every
// portion go into the convolution's ring (slots, behind and pos per row).
PK_API int pk_ssd_out(const PkStateMixer* d, const float* norm_w, int parts, float eps, const int* slots, const int* behind, const int* pos, int rows,
                      void* out, int ldo, int width, int out_f32, cudaStream_t stream) {
  if (!ssd_ok(d) || norm_w == nullptr || slots == nullptr || behind == nullptr || pos == nullptr || rows < 1 || rows > 65535 || out == nullptr || parts < 1 ||
      d->H * d->V % parts != 0 || width < d->H * d->V || ldo < width)
    return PK_ERR_BAD_ARG;
  const bool v4 = (d->H * d->V / parts & 3) == 0 && (d->ld & 3) == 0 && (d->og & 3) == 0 && ((uintptr_t)d->proj & 15) == 0 && ((uintptr_t)d->o & 15) == 0 &&
                  ((uintptr_t)norm_w & 15) == 0 && (ldo & 3) == 0 && ((uintptr_t)out & 15) == 0;
  float* f = (float*)out;
  pk::bf16* b = (pk::bf16*)out;
  if (v4) return out_f32 ? launch_out<float, 4>(*d, norm_w, parts, eps, slots, behind, pos, rows, f, ldo, width, stream)
                         : launch_out<pk::bf16, 4>(*d, norm_w, parts, eps, slots, behind, pos, rows, b, ldo, width, stream);
  return out_f32 ? launch_out<float, 1>(*d, norm_w, parts, eps, slots, behind, pos, rows, f, ldo, width, stream)
                 : launch_out<pk::bf16, 1>(*d, norm_w, parts, eps, slots, behind, pos, rows, b, ldo, width, stream);
}
