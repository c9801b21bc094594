// Prefill attention of long portions on the 5th-generation tensor cores, straight from the paged cache (paged_attention.cu
// describes the variants): grouped-query, causal, optional window or chunks, capped scores, a sink, one or two softmax maps per head.
//
// One CTA works one (head, tile of up to 128 query rows of one portion, slice of up to 128 value columns) and NMAP of the
// head's maps. A step is one page, 64 positions; its keys and values arrive by TMA (no multicast) into two alternating
// buffers each, the address of a page being its row in the pool. Per step and map:
//   S  = Q K^T       tcgen05.mma kind::f16, both operands K-major, fp32 S in TMEM (two buffers: S of the next step is
//                    computed while the softmax warps work on this one)
//   P  = exp2(S-m)   four softmax warps, one query row per thread; fp32 weights, handed to the tensor cores as the sum of two
//                    bf16 terms (16 significant bits)
//   O += P V         V as an MN-major operand, O in TMEM. The reference m of a row only moves when its maximum has grown by
//                    more than a factor of 2^8; its warp then rescales O in TMEM (weights up to 2^8 lose nothing in fp32)
// With NMAP = 2 the maps share the loads of V, and while one map's warps are in their exponentials the other map's products
// run; at the end the second map's warps hand lambda x their output through shared memory to the first map's, which take the
// difference, norm it over the head and store it. Heads too wide for that run one map per CTA and leave fp32 outputs for the
// merge kernel.
//
// Positions outside a row's view are masked; what a page holds behind the last position is finite (zeros or older rows).
// Every wait is bounded (status word + CTA-wide abort flag).
#include "../common/pk_paged.h"
#include "../common/pk_sm100.cuh"

namespace {

using namespace pk;
using namespace pk::sm100;

constexpr int kQ = 128;              // query rows of a tile
constexpr int kKV = 64;              // positions of a step = positions of a page
constexpr int kQPanel = kQ * 128;    // bytes of a 64-element-wide panel
constexpr int kKPanel = kKV * 128;

struct Params {
  PkPagedAttention a;
  const int4* tiles;       // {first step row, rows, portion, unused}
  const int4* seqs;        // {first step row, tokens, slot, first position}
  int qk_panels, k_steps;  // key width in 64-element panels and in 16-element products
  float scale_log2;
  float cap_in, cap_out;   // cap_in > 0: score x cap_in = 2 log2(e) score / cap; cap_out = cap log2(e)
  int raw;                 // outputs go to part_o [rows, H x maps, V]
};

struct Ctl {
  uint64_t q_full, k_full[2], k_empty[2], v_full[2], v_empty[2], s_full[2][2], p_ready[2], pv_full[2];
  uint32_t tmem_base;
  volatile uint32_t abort_flag;
};

// MN-major operand with the 128-byte swizzle (see attention_prefill.cu)
__device__ __forceinline__ uint64_t desc_mn_sw128(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3ffffu) >> 4);
  d |= (uint64_t)((lbo >> 4) & 0x3fffu) << 16;
  d |= (uint64_t)((sbo >> 4) & 0x3fffu) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

constexpr float kSlack = 8.f;        // log2 of how far a row's maximum may run ahead of its reference

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// y <- cap_out tanh(x / cap) from x cap_in, by tanh(u) = 1 - 2 / (exp(2 u) + 1): absolute error a few 2^-23 of the cap
__device__ __forceinline__ float soft_cap_log2(float x, float cap_in, float cap_out) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(exp2_approx(x * cap_in) + 1.f));
  return fmaf(-2.f * cap_out, r, cap_out);
}

template <int VP, int NMAP>    // value columns of this CTA's slice: 64 or 128; maps worked together
__global__ void __launch_bounds__(64 + 128 * NMAP, 1)
paged_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_c, const __grid_constant__ Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int NV = VP / 64;
  constexpr uint32_t kTmemCols = NMAP == 2 ? 512 : 256;
  const PkPagedAttention& a = p.a;
  const int qp = p.qk_panels;
  uint8_t* sp = base;                                   // [NMAP][2 terms] of 128 rows (1024-byte aligned panels throughout)
  uint8_t* sq = sp + NMAP * 2 * kQPanel;                // [NMAP][qp] panels of 128 rows
  uint8_t* sk = sq + NMAP * qp * kQPanel;               // [2][NMAP][qp] panels of 64 rows
  uint8_t* sv = sk + 2 * NMAP * qp * kKPanel;           // [2][NV]
  Ctl& ct = *reinterpret_cast<Ctl*>(sv + 2 * NV * kKPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vec0 = blockIdx.x * NMAP;                   // first query vector (head x maps + map)
  const int h = vec0 / a.maps, map0 = vec0 - h * a.maps, g = h / (a.H / a.G), vs = blockIdx.z;
  const int4 tile = p.tiles[gridDim.y - 1 - blockIdx.y];     // the last tiles of a portion see most: they go first
  const int4 seq = p.seqs[tile.z];
  const int pos0 = seq.w + tile.x - seq.x;              // position of the tile's first row
  int first = 0;
  if (a.window > 0) first = max(first, pos0 - a.window + 1);
  if (a.chunk > 0) first = max(first, pos0 / a.chunk * a.chunk);
  first = first / kKV * kKV;
  const int n_tiles = (pos0 + tile.y - 1 - first) / kKV + 1;

  if (threadIdx.x == 0) {
    mbar_init(&ct.q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&ct.k_full[i], 1);
      mbar_init(&ct.k_empty[i], 1);
      mbar_init(&ct.v_full[i], 1);
      mbar_init(&ct.v_empty[i], 1);
      mbar_init(&ct.s_full[i][0], 1);
      mbar_init(&ct.s_full[i][1], 1);
      mbar_init(&ct.p_ready[i], 4);
      mbar_init(&ct.pv_full[i], 1);
    }
    ct.abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 0) {
    tmem_alloc(&ct.tmem_base, kTmemCols);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_s = ct.tmem_base, tmem_o = ct.tmem_base + NMAP * 128;      // S [NMAP][2 buffers] of 64 columns, O [NMAP] of VP

  if (warp == 1) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      tma_prefetch_desc(&tmap_q);
      tma_prefetch_desc(&tmap_c);
      const int* pages = a.table + (size_t)seq.z * a.table_ld + first / kKV;
      const int kx = (g * a.maps + map0) * a.dp, vx = a.G * a.maps * a.dp + g * a.vp + vs * 128;
      mbar_arrive_expect_tx(&ct.q_full, NMAP * qp * kQPanel);
      for (int i = 0; i < NMAP * qp; ++i) {
        const int x = (vec0 + i / qp) * a.q_ld + (i % qp) * 64;
        tma_load_2d(sq + i * kQPanel, &tmap_q, &ct.q_full, x, tile.x);
        tma_load_2d(sq + i * kQPanel + kQPanel / 2, &tmap_q, &ct.q_full, x, tile.x + kQ / 2);
      }
      int k_issued = 0, v_issued = 0;
      int page = pages[0];
      for (int t = 0; t < n_tiles; ++t) {
        const int b = t & 1, y = page * kKV;
        if (t + 1 < n_tiles) page = pages[t + 1];
        if (t >= 2 && !mbar_wait(&ct.k_empty[b], ((t - 2) >> 1) & 1, &ct.abort_flag, a.status, 70)) break;
        mbar_arrive_expect_tx(&ct.k_full[b], NMAP * qp * kKPanel);
        for (int i = 0; i < NMAP * qp; ++i)
          tma_load_2d(sk + (b * NMAP * qp + i) * kKPanel, &tmap_c, &ct.k_full[b], kx + (i / qp) * a.dp + (i % qp) * 64, y);
        k_issued = t + 1;
        if (t >= 2 && !mbar_wait(&ct.v_empty[b], ((t - 2) >> 1) & 1, &ct.abort_flag, a.status, 71)) break;
        mbar_arrive_expect_tx(&ct.v_full[b], NV * kKPanel);
#pragma unroll
        for (int i = 0; i < NV; ++i) tma_load_2d(sv + (b * NV + i) * kKPanel, &tmap_c, &ct.v_full[b], vx + i * 64, y);
        v_issued = t + 1;
      }
      // every copy has landed before the CTA may exit, also when another warp gave up
      for (uint32_t i = 0; i < (1u << 20); ++i)
        if (mbar_try_wait(&ct.q_full, 0)) break;
      for (int t = max(k_issued - 2, 0); t < k_issued; ++t)
        for (uint32_t i = 0; i < (1u << 20); ++i)
          if (mbar_try_wait(&ct.k_full[t & 1], (t >> 1) & 1)) break;
      for (int t = max(v_issued - 2, 0); t < v_issued; ++t)
        for (uint32_t i = 0; i < (1u << 20); ++i)
          if (mbar_try_wait(&ct.v_full[t & 1], (t >> 1) & 1)) break;
    }
    __syncwarp();
  } else if (warp == 0) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc(1, 1, kQ, kKV);
      constexpr uint32_t idesc_pv = umma_idesc(1, 1, kQ, VP) | (1u << 16);   // V MN-major
      // S of step t for every map; its buffers were read two steps ago
      auto issue_s = [&](int t) {
        const int b = t & 1;
        for (int m = 0; m < NMAP; ++m) {
          const uint32_t qa = smem_u32(sq + m * qp * kQPanel), ka = smem_u32(sk + (b * NMAP + m) * qp * kKPanel);
          for (int j = 0; j < p.k_steps; ++j)
            umma_f16(tmem_s + m * 128 + b * 64, smem_desc_k_sw128(qa + (j >> 2) * kQPanel + (j & 3) * 32),
                     smem_desc_k_sw128(ka + (j >> 2) * kKPanel + (j & 3) * 32), idesc_s, j > 0 ? 1u : 0u);
          umma_commit(&ct.s_full[m][b]);
        }
        if (t + 2 < n_tiles) umma_commit(&ct.k_empty[b]);
      };
      bool ok = mbar_wait(&ct.q_full, 0, &ct.abort_flag, a.status, 72) && mbar_wait(&ct.k_full[0], 0, &ct.abort_flag, a.status, 73);
      if (ok) {
        tc_fence_after();
        issue_s(0);
      }
      for (int t = 0; t < n_tiles && ok; ++t) {
        const int b = t & 1;
        if (t + 1 < n_tiles) {
          // p_ready of step t - 1 was waited for: the S buffers of step t + 1 are free
          if (!mbar_wait(&ct.k_full[b ^ 1], ((t + 1) >> 1) & 1, &ct.abort_flag, a.status, 74)) break;
          tc_fence_after();
          issue_s(t + 1);
        }
        if (!mbar_wait(&ct.v_full[b], (t >> 1) & 1, &ct.abort_flag, a.status, 75)) break;
        for (int m = 0; m < NMAP; ++m) {
          if (!mbar_wait(&ct.p_ready[m], t & 1, &ct.abort_flag, a.status, 76)) {
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t pa = smem_u32(sp + m * 2 * kQPanel), va = smem_u32(sv + b * NV * kKPanel);
#pragma unroll
          for (int j = 0; j < 8; ++j)   // four k-steps of the leading bf16 term, then four of the remainder
            umma_f16(tmem_o + m * VP, smem_desc_k_sw128(pa + (j >> 2) * kQPanel + (j & 3) * 32), desc_mn_sw128(va + (j & 3) * 2048, kKPanel, 1024),
                     idesc_pv, t > 0 || j > 0 ? 1u : 0u);
          umma_commit(&ct.pv_full[m]);
        }
        if (ok && t + 2 < n_tiles) umma_commit(&ct.v_empty[b]);
      }
    }
    __syncwarp();
  } else {
    // ---------------- softmax ----------------
    const int m = (warp - 2) >> 2, q4 = warp & 3;
    const int r = q4 * 32 + lane;
    const int q_pos = pos0 + min(r, tile.y - 1);
    int lo = 0;
    if (a.window > 0) lo = max(lo, q_pos - a.window + 1);
    if (a.chunk > 0) lo = max(lo, q_pos / a.chunk * a.chunk);
    const uint32_t lane_off = (uint32_t)(q4 * 32) << 16;
    const uint32_t ts = tmem_s + m * 128 + lane_off, to = tmem_o + m * VP + lane_off;
    float ref = -INFINITY, sum = 0.f;      // the row's reference (log2 units) and the sum of its weights
    if (a.sink) {                          // the sink is the first score of every row
      ref = a.sink[vec0 + m] * 1.4426950408889634f;
      sum = 1.f;
    }
    const float to_log2 = p.cap_in > 0.f ? 1.f : p.scale_log2;
    bool ok = true;
    uint8_t* prow = sp + m * 2 * kQPanel + r * 128;
    for (int t = 0; t < n_tiles; ++t) {
      if (!mbar_wait_warp(&ct.s_full[m][t & 1], (t >> 1) & 1, &ct.abort_flag, a.status, 77)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t s[2][32];
      tmem_ld_32x32(ts + (t & 1) * 64, s[0]);
      tmem_ld_32x32(ts + (t & 1) * 64 + 32, s[1]);
      tmem_ld_wait();
      if (p.cap_in > 0.f) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i) s[c][i] = __float_as_uint(soft_cap_log2(__uint_as_float(s[c][i]), p.cap_in, p.cap_out));
      }
      // visible columns of this row in this step: [c_lo, c_hi]
      const int c_lo = lo - (first + t * kKV), c_hi = q_pos - (first + t * kKV);
      if (__any_sync(0xffffffffu, c_lo > 0 || c_hi < kKV - 1)) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < c_lo || c * 32 + i > c_hi) s[c][i] = 0xff800000u;
      }
      float t4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) t4[i & 3] = fmaxf(t4[i & 3], __uint_as_float(s[c][i]));
      const float top = fmaxf(fmaxf(t4[0], t4[1]), fmaxf(t4[2], t4[3])) * to_log2;
      bool waited = t == 0;
      if (ref == -INFINITY) ref = top;      // nothing was visible so far: sum and O are zero
      const bool grow = top > ref + kSlack;
      if (__any_sync(0xffffffffu, grow)) {
        const float alpha = grow ? exp2_approx(ref - top) : 1.f;
        if (t > 0) {
          if (!mbar_wait_warp(&ct.pv_full[m], (t - 1) & 1, &ct.abort_flag, a.status, 78)) {
            ok = false;
            break;
          }
          waited = true;
          tc_fence_after();
#pragma unroll 1
          for (int c = 0; c < VP / 32; ++c) {
            uint32_t x[32];
            tmem_ld_32x32(to + c * 32, x);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) x[i] = __float_as_uint(__uint_as_float(x[i]) * alpha);
            tmem_st_32x32(to + c * 32, x);
          }
          tmem_st_wait();
        }
        sum *= alpha;
        if (grow) ref = top;
      }
      const float mb = ref == -INFINITY ? 0.f : ref;
      float u4[4] = {0.f, 0.f, 0.f, 0.f};
      // weights as pairs: s[c][2e] <- leading terms, s[c][2e + 1] <- remainders
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float x = exp2_approx(fmaf(__uint_as_float(s[c][2 * e]), to_log2, -mb));
          const float y = exp2_approx(fmaf(__uint_as_float(s[c][2 * e + 1]), to_log2, -mb));
          u4[e & 3] += x + y;
          const __nv_bfloat162 ph = __floats2bfloat162_rn(x, y);
          const uint32_t hb = *reinterpret_cast<const uint32_t*>(&ph);
          const __nv_bfloat162 pl = __floats2bfloat162_rn(x - __uint_as_float(hb << 16), y - __uint_as_float(hb & 0xffff0000u));
          s[c][2 * e] = hb;
          s[c][2 * e + 1] = *reinterpret_cast<const uint32_t*>(&pl);
        }
      sum += (u4[0] + u4[1]) + (u4[2] + u4[3]);
      // the P buffers are free once the product of the step before is done
      if (!waited && !mbar_wait_warp(&ct.pv_full[m], (t - 1) & 1, &ct.abort_flag, a.status, 79)) {
        ok = false;
        break;
      }
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int gr = 0; gr < 4; ++gr) {
          const int piece = (c * 4 + gr) ^ (r & 7), e = gr * 8;
          *reinterpret_cast<uint4*>(prow + piece * 16) = make_uint4(s[c][e], s[c][e + 2], s[c][e + 4], s[c][e + 6]);
          *reinterpret_cast<uint4*>(prow + kQPanel + piece * 16) = make_uint4(s[c][e + 1], s[c][e + 3], s[c][e + 5], s[c][e + 7]);
        }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ct.p_ready[m]);
    }
    if (ok && !mbar_wait_warp(&ct.pv_full[m], (n_tiles - 1) & 1, &ct.abort_flag, a.status, 69)) ok = false;
    tc_fence_after();
    float inv = sum > 0.f ? 1.f / sum : 0.f;
    const bool row_ok = ok && r < tile.y;
    const int nv = min(VP, a.V - vs * 128);
    float* xch = reinterpret_cast<float*>(sp);          // [VP][128 rows]
    if (NMAP == 2) {
      // every product of this CTA is done once both groups have waited for their last one: the P buffers are free
      asm volatile("bar.sync 1, 256;" ::: "memory");
      if (m == 1) {
        inv *= a.lambda;
#pragma unroll 1
        for (int c = 0; c < VP / 32; ++c) {
          uint32_t x[32];
          tmem_ld_32x32(to + c * 32, x);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; ++i) xch[(c * 32 + i) * kQ + r] = __uint_as_float(x[i]) * inv;
        }
      }
      asm volatile("bar.sync 1, 256;" ::: "memory");
    }
    if (m == 0) {
      // columns c * 32 .. of this row's output (all lanes of the warp take part)
      auto output = [&](int c, float (&o)[32]) {
        uint32_t x[32];
        tmem_ld_32x32(to + c * 32, x);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          o[i] = __uint_as_float(x[i]) * inv;
          if (NMAP == 2) o[i] -= xch[(c * 32 + i) * kQ + r];
        }
      };
      float f = a.post;
      if (a.head_norm && !p.raw) {
        float ss = 0.f;
#pragma unroll 1
        for (int c = 0; c < VP / 32; ++c) {
          float o[32];
          output(c, o);
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < nv) ss = fmaf(o[i], o[i], ss);
        }
        f = a.post / sqrtf(ss / (float)a.V + a.eps);
      }
      if (a.gate >= 0 && !p.raw && row_ok) f /= 1.f + expf(-a.proj[(size_t)(tile.x + r) * a.ld + a.gate + h]);
#pragma unroll 1
      for (int c = 0; c < VP / 32; ++c) {
        float o[32];
        output(c, o);
        if (!row_ok) continue;
        if (p.raw) {
          float* dst = a.part_o + ((size_t)(tile.x + r) * a.H * a.maps + vec0) * a.V + vs * 128 + c * 32;
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < nv) dst[i] = o[i];
          continue;
        }
        bf16* dst = (bf16*)a.out + (size_t)(tile.x + r) * a.ldo + h * a.V + vs * 128 + c * 32;
        if ((a.V & 7) == 0) {
#pragma unroll
          for (int v = 0; v < 4; ++v) {
            if (c * 32 + v * 8 < nv) {
              uint32_t w[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) {
                const __nv_bfloat162 pr = __floats2bfloat162_rn(o[v * 8 + e * 2] * f, o[v * 8 + e * 2 + 1] * f);
                w[e] = *reinterpret_cast<const uint32_t*>(&pr);
              }
              *reinterpret_cast<uint4*>(dst + v * 8) = make_uint4(w[0], w[1], w[2], w[3]);
            }
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i < nv) dst[i] = __float2bfloat16(o[i] * f);
        }
      }
      if (row_ok && !p.raw && h == a.H - 1 && vs == 0)
        for (int i = a.H * a.V; i < a.width; ++i) ((bf16*)a.out)[(size_t)(tile.x + r) * a.ldo + i] = __float2bfloat16(0.f);
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    tmem_dealloc(ct.tmem_base, kTmemCols);
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

bool encode_rows64(EncodeTiledFn encode, CUtensorMap* map, const void* base, uint64_t cols, uint64_t rows) {
  const cuuint64_t gdim[2] = {cols, rows};
  const cuuint64_t gstride[1] = {cols * 2};
  const cuuint32_t box[2] = {64, 64};
  const cuuint32_t estr[2] = {1, 1};
  return encode(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), gdim, gstride, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

size_t smem_bytes(int qp, int vpan, int nmap) {
  return 1024 + (size_t)nmap * (2 + qp) * kQPanel + 2 * (size_t)(nmap * qp + vpan) * kKPanel + sizeof(Ctl);
}

template <int VP, int NMAP>
int launch(const CUtensorMap& tq, const CUtensorMap& tc, const Params& p, dim3 grid, cudaStream_t stream) {
  static PkDeviceOnce once;
  if (PkDeviceOnceGuard g{once}; g.needed()) {
    if (cudaFuncSetAttribute(paged_prefill_kernel<VP, NMAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    g.done();
  }
  paged_prefill_kernel<VP, NMAP><<<grid, 64 + 128 * NMAP, smem_bytes(p.qk_panels, VP / 64, NMAP), stream>>>(tq, tc, p);
  PK_CHECK_LAUNCH();
  return PK_OK;
}

}  // namespace

// 1 when the kernel writes finished outputs for this shape, 0 when it leaves fp32 outputs in part_o [rows, H x maps, V] for
// pk_paged_merge (nsplit 1, no part_ml), -1 when keys are too wide for it.
PK_API int pk_paged_prefill_form(int maps, int D, int V) {
  const int qp = (D + 63) / 64;
  if (qp > 4 || smem_bytes(qp, V <= 64 ? 1 : 2, 1) > 227 * 1024) return -1;
  if (V > 128) return 0;
  return maps == 1 || smem_bytes(qp, V <= 64 ? 1 : 2, 2) <= 227 * 1024 ? 1 : 0;
}

// Long portions (bf16): qf [rows, H x maps, q_ld] with q_ld a multiple of 64, cache of `pages` pages; tiles [ntiles] and seqs as in
// Params.
PK_API int pk_paged_prefill(const PkPagedAttention* a, int rows, int pages, const void* tiles, int ntiles, const void* seqs, cudaStream_t stream) {
  if (a == nullptr || a->f32 || rows < 1 || pages < 1 || ntiles < 1 || ntiles > 65535 || tiles == nullptr || seqs == nullptr || a->qf == nullptr || a->cache == nullptr)
    return PK_ERR_BAD_ARG;
  if (a->H < 1 || a->G < 1 || a->H % a->G != 0 || (a->maps != 1 && a->maps != 2) || a->D < 1 || a->V < 1 || a->V > 512 || a->V > a->vp) return PK_ERR_BAD_ARG;
  if (!(a->scale > 0.f)) return PK_ERR_UNSUPPORTED;      // masked scores are -inf before the scale
  if ((a->dp & 7) != 0 || a->dp < a->D || (a->vp & 7) != 0 || (a->row & 7) != 0 || a->row < a->G * (a->maps * a->dp + a->vp) || (a->q_ld & 63) != 0 ||
      a->q_ld < a->D)
    return PK_ERR_BAD_ARG;
  if (((uintptr_t)a->qf & 15) != 0 || ((uintptr_t)a->cache & 15) != 0) return PK_ERR_BAD_ARG;
  const int form = pk_paged_prefill_form(a->maps, a->D, a->V);
  if (form < 0) return PK_ERR_UNSUPPORTED;
  if (form == 0 ? a->part_o == nullptr : (a->out == nullptr || ((uintptr_t)a->out & 15) != 0 || (a->ldo & 7) != 0 || a->width < a->H * a->V || a->ldo < a->width ||
                                    (a->gate >= 0 && a->proj == nullptr)))
    return PK_ERR_BAD_ARG;
  EncodeTiledFn encode = encode_fn();
  if (encode == nullptr) return PK_ERR_UNSUPPORTED;
  CUtensorMap tq, tc;
  if (!encode_rows64(encode, &tq, a->qf, (uint64_t)a->H * a->maps * a->q_ld, (uint64_t)rows)) return PK_ERR_CUDA;
  if (!encode_rows64(encode, &tc, a->cache, (uint64_t)a->row, (uint64_t)pages * kKV)) return PK_ERR_CUDA;
  Params p{*a, (const int4*)tiles, (const int4*)seqs, (a->D + 63) / 64, (a->D + 15) / 16, a->scale * 1.4426950408889634f,
           a->cap > 0.f ? 2.f * 1.4426950408889634f * a->scale / a->cap : 0.f, a->cap * 1.4426950408889634f, form == 0 ? 1 : 0};
  const int slices = (a->V + 127) / 128;
  const bool narrow = a->V <= 64;
  if (form == 1 && a->maps == 2) return narrow ? launch<64, 2>(tq, tc, p, dim3(a->H, ntiles, 1), stream) : launch<128, 2>(tq, tc, p, dim3(a->H, ntiles, 1), stream);
  const dim3 grid(a->H * a->maps, ntiles, slices);
  return narrow ? launch<64, 1>(tq, tc, p, grid, stream) : launch<128, 1>(tq, tc, p, grid, stream);
}
