// Residual steps of decoders that norm behind the sum: one launch does everything between two sublayers,
//   x   <- embedding row + sinusoid of the position                (first layer)    or
//   x   <- rms(alpha x + sigmoid(g + b) * y) * w                   (y = the sublayer's output, g = its gate's logits; y may be the
//                                                                   sum of a few listed rows, the outputs of a token's experts,
//                                                                   and of a row of a second matrix, a shared expert's)
//   out <- x, and x + (x' - x) * shift                             (x' = the previous token's x; bf16 or fp32, columns padded)
//   or, behind the last layer, out <- rms(x) * w_out               (of listed rows)
// x is read from one buffer and written to another. A block works a few consecutive rows and carries x from row to row for the
// token shift; the row before its first one is computed again (its inputs are still there). At the start of a portion the previous
// x comes from the request's slot (zero at position 0); the x that a layer's shift will need is kept by the step that ends the
// layer's mixer, when every reader of the old one is done: it is that step's input row of a portion's last token.
#include "../common/pk_rotary.cuh"
#include "../common/pk_vec.cuh"

// Plain data mirrored by the Python bindings.
struct PkPostNorm {
  const float* x;          // [rows, width] (null: x starts from the embedding)
  float* x_out;            // [rows, width] (null: not kept)
  const int* tokens;
  const void* embed;       // [vocab, width] bf16
  const double* freq;      // [(width + 1) / 2] of the sinusoids (null: none)
  const float* y;          // [.., ldy]
  const int* y_rows;       // [rows, y_top]: y of a row is the sum of these rows (null: the row of the same index)
  const float* y2;         // [rows, ldy2] added to y (null: nothing)
  const float* gate;       // [rows, ldg] (null: no gate)
  const float* gate_b;     // [width]
  const float* w;          // [width]
  const float* w_out;      // [width] (null: out is x)
  const int* pos;
  const int* slot;
  const int* behind;       // tokens of the same portion after a row
  float* save;             // [slots, width] <- input row of every portion's last token (null: nothing is kept)
  const float* shift;      // [width] (null: no out_shift)
  const float* before;     // [slots, width] x of the token before a portion
  const int* rows;         // output row r works on row rows[r] (null: r)
  void* out;               // [M, ldo] (null: none)
  void* out_shift;         // [M, ldo]
  int vocab, ldy, y_top, ldy2, ldg, M, width, ldo, out_f32;
  float alpha, eps;
};

namespace {

using namespace pk;

// PT groups of VW values per thread. One group (few rows): the weights, which no kernel writes, are fetched before the wait. Several
// groups (many rows): they are read where they are used, which leaves registers for more blocks.
template <typename OutT, int PT, int VW, int THREADS, bool SHIFT>
__global__ void __launch_bounds__(THREADS, PT == 2 ? 2 : 1) post_norm_kernel(const PkPostNorm p, int per_block) {
  constexpr bool EARLY = PT == 1;
  pdl_trigger();
  __shared__ float scratch[33];
  const int tid = threadIdx.x, nt = blockDim.x;
  float wn[VW], gb[VW], sh[VW], prev[SHIFT ? PT : 1][VW];
#pragma unroll
  for (int j = 0; j < VW; ++j) wn[j] = gb[j] = sh[j] = 0.f;
  if (EARLY && tid * VW < p.width) {
    if (p.w) load_f32<VW>(p.w + tid * VW, wn);
    if (p.gate) load_f32<VW>(p.gate_b + tid * VW, gb);
    if (SHIFT) load_f32<VW>(p.shift + tid * VW, sh);
  }
  pdl_wait();
  const int r0 = blockIdx.x * per_block, r1 = min(r0 + per_block, p.M);
  const bool again = SHIFT && r0 > 0 && p.behind[r0 - 1] > 0;      // the row before is of the same portion
  for (int r = r0 - (again ? 1 : 0); r < r1; ++r) {
    const bool own = r >= r0;
    const int row = p.rows ? p.rows[r] : r;
    float v[PT][VW];
#pragma unroll
    for (int i = 0; i < PT; ++i)
#pragma unroll
      for (int j = 0; j < VW; ++j) v[i][j] = 0.f;
    if (p.x == nullptr) {
      int t = p.tokens[row];
      t = t < 0 ? 0 : (t >= p.vocab ? p.vocab - 1 : t);
      const int pos = p.pos[row];
#pragma unroll
      for (int i = 0; i < PT; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= p.width) continue;
        load_any<VW>(p.embed, (size_t)t * p.width + c, false, v[i]);
        if (p.freq) {
          if (VW == 4) {
#pragma unroll
            for (int j = 0; j < VW; j += 2) {
              float s, co;
              rotary_sincos(p.freq[(c + j) >> 1], pos, s, co);
              v[i][j] += s;
              v[i][(j + 1) % VW] += co;
            }
          } else {
            float s, co;
            rotary_sincos(p.freq[c >> 1], pos, s, co);
            v[i][0] += (c & 1) ? co : s;
          }
        }
      }
    } else {
      const size_t at = (size_t)row * p.width;
      const bool keep = own && p.save && p.behind[row] == 0;
      // all loads of a row are in flight together
      float u[PT][VW], g[PT][VW];
#pragma unroll
      for (int i = 0; i < PT; ++i) {
        const int c = (tid + i * nt) * VW;
#pragma unroll
        for (int j = 0; j < VW; ++j) u[i][j] = g[i][j] = 0.f;
        if (c >= p.width) continue;
        load_f32<VW>(p.x + at + c, v[i]);
        if (p.gate) load_f32<VW>(p.gate + (size_t)row * p.ldg + c, g[i]);
        if (!p.y_rows) load_f32<VW>(p.y + (size_t)row * p.ldy + c, u[i]);
      }
      auto add_row = [&](const float* y) {
        float a[PT][VW];
#pragma unroll
        for (int i = 0; i < PT; ++i) {
#pragma unroll
          for (int j = 0; j < VW; ++j) a[i][j] = 0.f;
          if ((tid + i * nt) * VW < p.width) load_f32<VW>(y + (tid + i * nt) * VW, a[i]);
        }
#pragma unroll
        for (int i = 0; i < PT; ++i)
#pragma unroll
          for (int j = 0; j < VW; ++j) u[i][j] += a[i][j];
      };
      if (p.y_rows) {
        const int* from = p.y_rows + (size_t)row * p.y_top;
        for (int k = 0; k < p.y_top; k += 2) {
          const int f0 = from[k], f1 = k + 1 < p.y_top ? from[k + 1] : -1;
          if (f0 >= 0) add_row(p.y + (size_t)f0 * p.ldy);
          if (f1 >= 0) add_row(p.y + (size_t)f1 * p.ldy);
        }
      }
      if (p.y2) add_row(p.y2 + (size_t)row * p.ldy2);
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < PT; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= p.width) continue;
        if (keep) store<VW>(p.save + (size_t)p.slot[row] * p.width + c, v[i]);
        if (!EARLY && p.gate) load_f32<VW>(p.gate_b + c, gb);
#pragma unroll
        for (int j = 0; j < VW; ++j) {
          const float f = p.gate ? 1.f / (1.f + expf(-(g[i][j] + gb[j]))) : 1.f;
          v[i][j] = fmaf(p.alpha, v[i][j], f * u[i][j]);
          ss = fmaf(v[i][j], v[i][j], ss);
        }
      }
      const float rr = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
#pragma unroll
      for (int i = 0; i < PT; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= p.width) continue;
        if (!EARLY) load_f32<VW>(p.w + c, wn);
#pragma unroll
        for (int j = 0; j < VW; ++j) v[i][j] = v[i][j] * rr * wn[j];
      }
    }
    if (own) {
      float rr = 1.f;
      if (p.w_out) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < PT; ++i)
#pragma unroll
          for (int j = 0; j < VW; ++j) ss = fmaf(v[i][j], v[i][j], ss);
        rr = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
      }
      const float* from = nullptr;      // x of the token before, when it is not carried
      const bool first = SHIFT && (r == 0 || p.behind[r - 1] == 0);
      if (first && p.pos[row] > 0) from = p.before + (size_t)p.slot[row] * p.width;
#pragma unroll
      for (int i = 0; i < PT; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= p.width) continue;
        if (p.x_out) store<VW>(p.x_out + (size_t)row * p.width + c, v[i]);
        if (p.out) {
          float o[VW];
          if (p.w_out) load_f32<VW>(p.w_out + c, o);
#pragma unroll
          for (int j = 0; j < VW; ++j) o[j] = p.w_out ? v[i][j] * rr * o[j] : v[i][j];
          store<VW>(reinterpret_cast<OutT*>(p.out) + (size_t)r * p.ldo + c, o);
        }
        if (SHIFT) {
          float o[VW];
          if (!EARLY) load_f32<VW>(p.shift + c, sh);
          if (first) {
#pragma unroll
            for (int j = 0; j < VW; ++j) prev[i][j] = 0.f;
            if (from) load_f32<VW>(from + c, prev[i]);
          }
#pragma unroll
          for (int j = 0; j < VW; ++j) o[j] = fmaf(prev[i][j] - v[i][j], sh[j], v[i][j]);
          store<VW>(reinterpret_cast<OutT*>(p.out_shift) + (size_t)r * p.ldo + c, o);
        }
      }
      for (int c = p.width + tid; c < p.ldo; c += nt) {
        if (p.out) reinterpret_cast<OutT*>(p.out)[(size_t)r * p.ldo + c] = (OutT)0.f;
        if (SHIFT) reinterpret_cast<OutT*>(p.out_shift)[(size_t)r * p.ldo + c] = (OutT)0.f;
      }
    }
    if (SHIFT) {
#pragma unroll
      for (int i = 0; i < PT; ++i)
#pragma unroll
        for (int j = 0; j < VW; ++j) prev[i][j] = v[i][j];
    }
  }
}

template <typename OutT, int VW, bool SHIFT>
int launch_norm(const PkPostNorm& p, cudaStream_t stream) {
  const int groups = (p.width + VW - 1) / VW;
  // few rows: as many threads as help their latency; many rows: two groups per thread, and a few rows per block so that fewer rows are
  // computed twice
  const int want = groups > 1024 ? 512 : p.M <= 64 ? groups : (groups + 1) / 2;
  const int nt = (want + 31) / 32 * 32;
  const int per = (groups + nt - 1) / nt;
  int rows = SHIFT ? p.M / 592 : 1;
  rows = rows < 1 ? 1 : rows > 4 ? 4 : rows;
  const dim3 grid((p.M + rows - 1) / rows);
#define PK_NORM_CASE(n, threads)                                                                                            \
  if (per <= n && nt <= threads) {                                                                                          \
    PK_LAUNCH_PDL((post_norm_kernel<OutT, n, VW, threads, SHIFT>), grid, dim3(nt), (size_t)0, stream, p, rows);             \
    return PK_OK;                                                                                                           \
  }
  PK_NORM_CASE(1, 256)
  PK_NORM_CASE(1, 1024)
  PK_NORM_CASE(2, 512)
  PK_NORM_CASE(4, 512)
  PK_NORM_CASE(8, 512)
  PK_NORM_CASE(16, 512)
#undef PK_NORM_CASE
  return PK_ERR_UNSUPPORTED;
}

template <typename OutT, int VW>
int launch_norm(const PkPostNorm& p, cudaStream_t stream) {
  return p.shift ? launch_norm<OutT, VW, true>(p, stream) : launch_norm<OutT, VW, false>(p, stream);
}

bool aligned(const void* p, int ld = 0) { return ((uintptr_t)p & 15) == 0 && (ld & 3) == 0; }

template <typename OutT>
int launch_any(const PkPostNorm& p, cudaStream_t stream) {
  const bool v4 = (p.width & 3) == 0 && aligned(p.x) && aligned(p.x_out) && aligned(p.embed) && aligned(p.y, p.ldy) && aligned(p.y2, p.y2 ? p.ldy2 : 0) &&
                  aligned(p.gate, p.gate ? p.ldg : 0) && aligned(p.gate_b) && aligned(p.w) && aligned(p.w_out) && aligned(p.save) && aligned(p.shift) &&
                  aligned(p.before) && aligned(p.out, p.ldo) && aligned(p.out_shift);
  return v4 ? launch_norm<OutT, 4>(p, stream) : launch_norm<OutT, 1>(p, stream);
}

}  // namespace

// See the head of this file. With a shift, rows are all rows of the step in order. width up to 8192 (32768 when a multiple of 4).
PK_API int pk_post_norm(const PkPostNorm* d, cudaStream_t stream) {
  if (d == nullptr || d->M < 1 || d->width < 1) return PK_ERR_BAD_ARG;
  if (d->x == nullptr && (d->tokens == nullptr || d->embed == nullptr || d->vocab < 1 || d->pos == nullptr)) return PK_ERR_BAD_ARG;
  if (d->x != nullptr && (d->y == nullptr || d->w == nullptr || d->ldy < d->width || (d->y_rows != nullptr && d->y_top < 1) || d->x == d->x_out)) return PK_ERR_BAD_ARG;
  if (d->y2 != nullptr && d->ldy2 < d->width) return PK_ERR_BAD_ARG;
  if (d->gate != nullptr && (d->gate_b == nullptr || d->ldg < d->width)) return PK_ERR_BAD_ARG;
  if (d->save != nullptr && (d->behind == nullptr || d->slot == nullptr)) return PK_ERR_BAD_ARG;
  if (d->shift != nullptr && (d->out_shift == nullptr || d->before == nullptr || d->behind == nullptr || d->slot == nullptr || d->pos == nullptr || d->rows != nullptr))
    return PK_ERR_BAD_ARG;
  if ((d->out != nullptr || d->out_shift != nullptr) && d->ldo < d->width) return PK_ERR_BAD_ARG;
  return d->out_f32 ? launch_any<float>(*d, stream) : launch_any<pk::bf16>(*d, stream);
}
