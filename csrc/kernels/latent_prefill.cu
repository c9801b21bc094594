// Prefill attention of long portions on the 5th-generation tensor cores, for latent attention with expanded keys and
// values (and any attention whose keys and values lie in contiguous rows): causal, optional sliding window, optional
// learned sink per head, optional sigmoid gate on the outputs, key width a multiple of 64 up to 256, value width a multiple of 64 in slices of up to 128.
//
// One CTA works one (head, tile of up to 128 query rows of one portion, slice of the value dim). For every 64 positions
// between the window's first and the causal limit:
//   S  = Q K^T      tcgen05.mma kind::f16, both operands K-major, fp32 S in TMEM
//   P  = exp2(S-m)  four softmax warps, one query row per thread; fp32 weights, handed to the tensor cores as the sum of
//                   two bf16 terms (16 significant bits)
//   PV = P V        V as an MN-major operand; the product of tile t runs together with S of tile t + 1
//   O  = O alpha + PV in fp32 registers
// K and V tiles arrive by TMA (no multicast) into two alternating buffers. Rows behind a portion's last position belong to
// the next portion or are zero-filled, and are masked. Every wait is bounded (status word + CTA-wide abort flag).
#include "../common/pk_sm100.cuh"

namespace {

using namespace pk;
using namespace pk::sm100;

constexpr int kQ = 128;              // query rows of a tile
constexpr int kKV = 64;              // positions of a step
constexpr int kQPanel = kQ * 128;    // bytes of a 64-element-wide panel
constexpr int kKPanel = kKV * 128;
constexpr int kThreads = 32 + 128;
constexpr uint32_t kTmemCols = 256;

struct Params {
  const int4* tiles;       // {first step row, rows, portion, unused}
  const int4* seqs;        // {first step row, tokens, slot, first position}
  const int2* gather;      // {first key row, its position}
  int H, qk_panels, v_panels_total, V, window;
  float scale_log2;
  const float* sink;       // [H] or null
  bf16* out;               // [rows, ldo]
  int ldo;
  const float* gate;       // [rows, ldg] logits of a sigmoid gate on the outputs, head h at h V (null: none)
  int ldg;
  uint32_t* status;
};

struct Ctl {
  uint64_t q_full, kv_full[2], s_full, p_ready, pv_full;
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

template <int VP>    // value columns of this CTA's slice: 64 or 128
__global__ void __launch_bounds__(kThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_kv, const Params p) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* base = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int NV = VP / 64;
  const int qp = p.qk_panels;
  uint8_t* sq = base;                                   // [qp] panels of 128 rows
  uint8_t* sk = sq + qp * kQPanel;                      // [2][qp] panels of 64 rows
  uint8_t* sv = sk + 2 * qp * kKPanel;                  // [2][NV]
  uint8_t* sp = sv + 2 * NV * kKPanel;                  // [2 terms] of 128 rows
  Ctl& ct = *reinterpret_cast<Ctl*>(sp + 2 * kQPanel);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, vs = blockIdx.z;
  const int4 tile = p.tiles[blockIdx.x];
  const int4 seq = p.seqs[tile.z];
  const int2 ga = p.gather[tile.z];
  const int pos0 = seq.w + tile.x - seq.x;              // position of the tile's first row
  const int first = p.window > 0 ? max(pos0 - p.window + 1, ga.y) : ga.y;
  const int n_tiles = (pos0 + tile.y - 1 - first) / kKV + 1;

  if (threadIdx.x == 0) {
    mbar_init(&ct.q_full, 1);
    mbar_init(&ct.kv_full[0], 1);
    mbar_init(&ct.kv_full[1], 1);
    mbar_init(&ct.s_full, 1);
    mbar_init(&ct.p_ready, 4);
    mbar_init(&ct.pv_full, 1);
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
  const uint32_t tmem_s = ct.tmem_base, tmem_pv = ct.tmem_base + 64;

  if (warp == 0) {
    if (lane == 0) {
      tma_prefetch_desc(&tmap_q);
      tma_prefetch_desc(&tmap_kv);
      const int y0 = ga.x + (first - ga.y);
      const int vx = (p.H * qp + h * p.v_panels_total + vs * 2) * 64;
      auto load_kv = [&](int t) {
        const int b = t & 1;
        mbar_arrive_expect_tx(&ct.kv_full[b], (qp + NV) * kKPanel);
        const int y = y0 + t * kKV;
        for (int i = 0; i < qp; ++i) tma_load_2d(sk + (b * qp + i) * kKPanel, &tmap_kv, &ct.kv_full[b], (h * qp + i) * 64, y);
#pragma unroll
        for (int i = 0; i < NV; ++i) tma_load_2d(sv + (b * NV + i) * kKPanel, &tmap_kv, &ct.kv_full[b], vx + i * 64, y);
      };
      mbar_arrive_expect_tx(&ct.q_full, qp * kQPanel);
      for (int i = 0; i < qp; ++i) {
        tma_load_2d(sq + i * kQPanel, &tmap_q, &ct.q_full, (h * qp + i) * 64, tile.x);
        tma_load_2d(sq + i * kQPanel + kQPanel / 2, &tmap_q, &ct.q_full, (h * qp + i) * 64, tile.x + kQ / 2);
      }
      int issued = 0;
      for (; issued < 2 && issued < n_tiles; ++issued) load_kv(issued);
      constexpr uint32_t idesc_s = umma_idesc(1, 1, kQ, kKV);
      constexpr uint32_t idesc_pv = umma_idesc(1, 1, kQ, VP) | (1u << 16);   // V MN-major
      auto issue_s = [&](int t) {
        const uint32_t qa = smem_u32(sq), ka = smem_u32(sk + (t & 1) * qp * kKPanel);
        for (int j = 0; j < qp * 4; ++j)
          umma_f16(tmem_s, smem_desc_k_sw128(qa + (j >> 2) * kQPanel + (j & 3) * 32),
                   smem_desc_k_sw128(ka + (j >> 2) * kKPanel + (j & 3) * 32), idesc_s, j > 0 ? 1u : 0u);
        umma_commit(&ct.s_full);
      };
      bool ok = mbar_wait(&ct.q_full, 0, &ct.abort_flag, p.status, 61) && mbar_wait(&ct.kv_full[0], 0, &ct.abort_flag, p.status, 62);
      bool q_landed = ok;
      if (ok) {
        tc_fence_after();
        issue_s(0);
      }
      for (int t = 0; t < n_tiles && ok; ++t) {
        const int b = t & 1;
        if (t + 1 < n_tiles && !mbar_wait(&ct.kv_full[b ^ 1], ((t + 1) >> 1) & 1, &ct.abort_flag, p.status, 63)) { ok = false; break; }
        if (!mbar_wait(&ct.p_ready, t & 1, &ct.abort_flag, p.status, 64)) { ok = false; break; }
        tc_fence_after();
        const uint32_t pa = smem_u32(sp), va = smem_u32(sv + b * NV * kKPanel);
#pragma unroll
        for (int j = 0; j < 8; ++j)   // four k-steps of the leading bf16 term, then four of the remainder
          umma_f16(tmem_pv, smem_desc_k_sw128(pa + (j >> 2) * kQPanel + (j & 3) * 32), desc_mn_sw128(va + (j & 3) * 2048, kKPanel, 1024), idesc_pv,
                   j > 0 ? 1u : 0u);
        umma_commit(&ct.pv_full);
        if (t + 1 < n_tiles) issue_s(t + 1);     // S of tile t was read before p_ready
        if (!mbar_wait(&ct.pv_full, t & 1, &ct.abort_flag, p.status, 65)) { ok = false; break; }
        if (issued < n_tiles) load_kv(issued++); // tile t's buffers are free: its S and PV products are done
      }
      if (!ok) {
        // gave up: let the loads in flight land before the CTA exits
        if (!q_landed)
          for (uint32_t i = 0; i < (1u << 20); ++i)
            if (mbar_try_wait(&ct.q_full, 0)) break;
        for (int t = max(issued - 2, 0); t < issued; ++t)
          for (uint32_t i = 0; i < (1u << 20); ++i)
            if (mbar_try_wait(&ct.kv_full[t & 1], (t >> 1) & 1)) break;
      }
    }
    __syncwarp();
  } else {
    const int q4 = warp & 3;
    const int r = q4 * 32 + lane;
    const bool row_ok = r < tile.y;
    const int q_pos = pos0 + min(r, tile.y - 1);
    const int lo = p.window > 0 ? q_pos - p.window + 1 : 0;
    const uint32_t lane_off = (uint32_t)(q4 * 32) << 16;
    float o[VP];
#pragma unroll
    for (int i = 0; i < VP; ++i) o[i] = 0.f;
    float mx = -INFINITY, sum = 0.f;
    bool ok = true;
    for (int t = 0; t < n_tiles && ok; ++t) {
      if (!mbar_wait(&ct.s_full, t & 1, &ct.abort_flag, p.status, 66)) { ok = false; break; }
      tc_fence_after();
      const int kv0 = first + t * kKV;
      uint32_t s[2][32];
      tmem_ld_32x32(tmem_s + lane_off, s[0]);
      tmem_ld_32x32(tmem_s + lane_off + 32, s[1]);
      tmem_ld_wait();
      float tmax = -INFINITY;
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          const int kp = kv0 + c * 32 + i;
          const float v = kp <= q_pos && kp >= lo ? __uint_as_float(s[c][i]) * p.scale_log2 : -INFINITY;
          s[c][i] = __float_as_uint(v);
          tmax = fmaxf(tmax, v);
        }
      const float m_new = fmaxf(mx, tmax);
      const float alpha = mx == -INFINITY ? 0.f : exp2f(mx - m_new);
      const float mb = m_new == -INFINITY ? 0.f : m_new;
      float tsum = 0.f;
      uint8_t* prow = sp + r * 128;
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int g = 0; g < 4; ++g) {
          uint32_t hi[4], lw[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float a = exp2f(__uint_as_float(s[c][g * 8 + e * 2]) - mb), b = exp2f(__uint_as_float(s[c][g * 8 + e * 2 + 1]) - mb);
            tsum += a + b;
            const __nv_bfloat162 ph = __floats2bfloat162_rn(a, b);
            const __nv_bfloat162 pl = __floats2bfloat162_rn(a - __bfloat162float(ph.x), b - __bfloat162float(ph.y));
            hi[e] = *reinterpret_cast<const uint32_t*>(&ph);
            lw[e] = *reinterpret_cast<const uint32_t*>(&pl);
          }
          const int chunk = (c * 4 + g) ^ (r & 7);
          *reinterpret_cast<uint4*>(prow + chunk * 16) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(prow + kQPanel + chunk * 16) = make_uint4(lw[0], lw[1], lw[2], lw[3]);
        }
      sum = sum * alpha + tsum;
      mx = m_new;
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&ct.p_ready);
      if (!mbar_wait(&ct.pv_full, t & 1, &ct.abort_flag, p.status, 67)) { ok = false; break; }
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < VP / 32; ++c) {
        uint32_t pv[32];
        tmem_ld_32x32(tmem_pv + lane_off + c * 32, pv);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 32; ++i) o[c * 32 + i] = fmaf(o[c * 32 + i], alpha, __uint_as_float(pv[i]));
      }
      tc_fence_before();
    }
    if (ok && row_ok) {
      float top = mx;
      float den = sum;
      float f = 1.f;
      if (p.sink) {
        const float s2 = p.sink[h] * 1.4426950408889634f;
        top = fmaxf(mx, s2);
        f = mx == -INFINITY ? 0.f : exp2f(mx - top);
        den = sum * f + exp2f(s2 - top);
      }
      const float inv = den > 0.f ? f / den : 0.f;
      bf16* dst = p.out + (size_t)(tile.x + r) * p.ldo + h * p.V + vs * 128;
      const int nv = min(VP, p.V - vs * 128);
#pragma unroll
      for (int v = 0; v < VP; ++v) o[v] *= inv;
      if (p.gate) {
        const float* g = p.gate + (size_t)(tile.x + r) * p.ldg + h * p.V + vs * 128;
        if ((p.V & 3) == 0 && (p.ldg & 3) == 0 && ((uintptr_t)p.gate & 15) == 0) {
#pragma unroll
          for (int v = 0; v < VP / 4; ++v)
            if (v * 4 < nv) {
              const float4 x = *reinterpret_cast<const float4*>(g + v * 4);
              o[v * 4] /= 1.f + __expf(-x.x);
              o[v * 4 + 1] /= 1.f + __expf(-x.y);
              o[v * 4 + 2] /= 1.f + __expf(-x.z);
              o[v * 4 + 3] /= 1.f + __expf(-x.w);
            }
        } else {
#pragma unroll
          for (int v = 0; v < VP; ++v)
            if (v < nv) o[v] /= 1.f + __expf(-g[v]);
        }
      }
      if ((p.V & 7) == 0) {
#pragma unroll
        for (int v = 0; v < VP / 8; ++v) {
          if (v * 8 < nv) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const __nv_bfloat162 pr = __floats2bfloat162_rn(o[v * 8 + e * 2], o[v * 8 + e * 2 + 1]);
              w[e] = *reinterpret_cast<const uint32_t*>(&pr);
            }
            *reinterpret_cast<uint4*>(dst + v * 8) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      } else {
#pragma unroll
        for (int v = 0; v < VP; ++v)
          if (v < nv) dst[v] = __float2bfloat16(o[v]);
      }
      if (h == p.H - 1 && vs == 0)
        for (int i = p.H * p.V; i < p.ldo; ++i) p.out[(size_t)(tile.x + r) * p.ldo + i] = __float2bfloat16(0.f);
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

template <int VP>
int launch(const CUtensorMap& tq, const CUtensorMap& tkv, const Params& p, dim3 grid, cudaStream_t stream) {
  const size_t smem = 1024 + (size_t)p.qk_panels * kQPanel + 2 * (size_t)(p.qk_panels + VP / 64) * kKPanel + 2 * kQPanel + sizeof(Ctl);
  if (smem > 227 * 1024) return PK_ERR_UNSUPPORTED;
  static PkDeviceOnce once;
  if (PkDeviceOnceGuard once_guard{once}; once_guard.needed()) {
    if (cudaFuncSetAttribute(latent_prefill_kernel<VP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) {
      pk_set_last_cuda_error((int)cudaGetLastError());
      return PK_ERR_CUDA;
    }
    once_guard.done();
  }
  latent_prefill_kernel<VP><<<grid, kThreads, smem, stream>>>(tq, tkv, p);
  PK_CHECK_LAUNCH();
  return PK_OK;
}

}  // namespace

// q [rows, H, qk_panels * 64] bf16; kv [kv_rows, H * qk_panels * 64 | H * v_panels * 64] bf16; tiles [ntiles], seqs, gather
// as in Params; out [rows, ldo] bf16, head h at h * V; gate [rows, ldg] or null. window <= 0: full causal.
PK_API int pk_latent_prefill(const void* q, int rows, const void* kv, int kv_rows, const void* tiles, int ntiles, const void* seqs,
                             const void* gather, int H, int qk_panels, int v_panels, int V, int window, float scale, const float* sink,
                             void* out, int ldo, const float* gate, int ldg, uint32_t* status, cudaStream_t stream) {
  if ((gate != nullptr && ldg < H * V) || rows < 1 || kv_rows < 1 || ntiles < 1 || H < 1 || V < 1 || V > v_panels * 64 || ldo < H * V || (ldo & 7) != 0) return PK_ERR_BAD_ARG;
  if (qk_panels < 1 || qk_panels > 4 || v_panels < 1) return PK_ERR_UNSUPPORTED;
  if (((uintptr_t)q & 15) != 0 || ((uintptr_t)kv & 15) != 0 || ((uintptr_t)out & 15) != 0) return PK_ERR_BAD_ARG;
  if (v_panels > 1 && (v_panels & 1) != 0) return PK_ERR_UNSUPPORTED;
  EncodeTiledFn encode = encode_fn();
  if (encode == nullptr) return PK_ERR_UNSUPPORTED;
  CUtensorMap tq, tkv;
  if (!encode_rows64(encode, &tq, q, (uint64_t)H * qk_panels * 64, (uint64_t)rows)) return PK_ERR_CUDA;
  if (!encode_rows64(encode, &tkv, kv, (uint64_t)H * (qk_panels + v_panels) * 64, (uint64_t)kv_rows)) return PK_ERR_CUDA;
  Params p{(const int4*)tiles, (const int4*)seqs, (const int2*)gather, H, qk_panels, v_panels, V, window, scale * 1.4426950408889634f, sink,
           (pk::bf16*)out, ldo, gate, ldg, status};
  if (v_panels == 1) return launch<64>(tq, tkv, p, dim3(ntiles, H, 1), stream);
  return launch<128>(tq, tkv, p, dim3(ntiles, H, v_panels / 2), stream);
}
