// Residual and norm steps of decoders whose residual stream is kept in fp32: one launch does everything between two
// projections,
//   x   <- scale * embedding row            (first layer)    or
//   x   <- x + rms(y) * (bias + w_post)     (y = the sublayer's output, fp32; no w_post: y as it is; y may be the sum of a
//                                            few listed rows, the outputs of a token's experts, and of another row times
//                                            a factor; a constant may multiply the whole term)
//   x   <- x + scale * embedding row        (again, before a further pass over the same layers)
//   out <- rms(x) * (bias + w_pre)          (the next sublayer's input, bf16 or fp32, columns padded with zeros)
// `bias` is 1 for weights stored around zero and 0 for plain weights. One block per row, the row stays in registers.
#include "../common/pk_vec.cuh"

namespace {

using namespace pk;

struct NormParams {
  float* x;              // [rows of the step, width] residual stream
  const int* tokens;     // embedding ids, or null
  const bf16* embed;
  int vocab;
  float embed_scale;
  int embed_add;         // 0: x starts as the embedding row; 1: the row is added to x (after y)
  const float* y;        // [rows, ldy] or null
  int ldy;
  const int* y_rows;     // [rows, y_top]: y of a row is the sum of these rows of `y` (null: the row of the same index)
  int y_top;               // (a negative entry stands for no row)
  float y_scale;           // factor on what is added
  const void* skip;        // [rows, ld_skip] or null: y of a row gets skip_w[row] x this row
  const float* skip_w;
  int ld_skip, skip_f32;
  const float* w_post;
  const int* rows;       // output row r works on residual row rows[r] (null: r); x is not written then
  int width;
  const float* w_pre;    // null: no output
  float bias, eps;
  void* out;             // [M, ldo]
  int ldo;
};

// A thread holds PT groups of VW adjacent values of its row (VW = 4 when width and strides allow 16-byte accesses).
template <typename OutT, int PT, int VW>
__global__ void __launch_bounds__(1024) sandwich_norm_kernel(const NormParams p) {
  pdl_trigger();
  __shared__ float scratch[33];
  const int r = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  // the norm weights are not written by any kernel: fetched before the wait
  float wb[PT][VW], wa[PT][VW];
#pragma unroll
  for (int i = 0; i < PT; ++i) {
    const int c = (tid + i * nt) * VW;
    if (c < p.width) {
      if (p.w_post) load_f32<VW>(p.w_post + c, wb[i]);
      if (p.w_pre) load_f32<VW>(p.w_pre + c, wa[i]);
    }
  }
  pdl_wait();
  const int row = p.rows ? p.rows[r] : r;
  float* xr = p.x + (size_t)row * p.width;
  float v[PT][VW], u[PT][VW];
  auto add_embedding = [&]() {
    int t = p.tokens[row];
    t = t < 0 ? 0 : (t >= p.vocab ? p.vocab - 1 : t);
    const bf16* e = p.embed + (size_t)t * p.width;
#pragma unroll
    for (int i = 0; i < PT; ++i)
#pragma unroll
      for (int j = 0; j < VW; ++j) {
        const int c = (tid + i * nt) * VW + j;
        if (c < p.width) v[i][j] = __fadd_rn(v[i][j], __fmul_rn(__bfloat162float(e[c]), p.embed_scale));
      }
  };
  const bool fresh = p.tokens && !p.embed_add;
#pragma unroll
  for (int i = 0; i < PT; ++i) {
    const int c = (tid + i * nt) * VW;
#pragma unroll
    for (int j = 0; j < VW; ++j) v[i][j] = 0.f;
    if (!fresh && c < p.width) load_f32<VW>(xr + c, v[i]);
  }
  if (fresh) add_embedding();
  if (p.y) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PT; ++i) {
      const int c = (tid + i * nt) * VW;
#pragma unroll
      for (int j = 0; j < VW; ++j) u[i][j] = 0.f;
      if (c < p.width) {
        if (p.y_rows) {
          for (int k = 0; k < p.y_top; ++k) {
            float a[VW];
            const int from = p.y_rows[(size_t)row * p.y_top + k];
            if (from < 0) continue;
            load_f32<VW>(p.y + (size_t)from * p.ldy + c, a);
#pragma unroll
            for (int j = 0; j < VW; ++j) u[i][j] += a[j];
          }
        } else {
          load_f32<VW>(p.y + (size_t)row * p.ldy + c, u[i]);
        }
        if (p.skip) {      // may be the buffer of `out`: this thread alone reads and later writes these columns
          const float f = p.skip_w[row];
          float a[VW];
          load_any<VW>(p.skip, (size_t)row * p.ld_skip + c, p.skip_f32, a);
          if (f != 0.f) {
#pragma unroll
            for (int j = 0; j < VW; ++j) u[i][j] = fmaf(f, a[j], u[i][j]);
          }
        }
      }
#pragma unroll
      for (int j = 0; j < VW; ++j) ss = fmaf(u[i][j], u[i][j], ss);
    }
    if (p.w_post) {
      const float rr = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
#pragma unroll
      for (int i = 0; i < PT; ++i)
        if ((tid + i * nt) * VW < p.width) {
#pragma unroll
          for (int j = 0; j < VW; ++j) v[i][j] += u[i][j] * rr * (p.bias + wb[i][j]) * p.y_scale;
        }
    } else {
#pragma unroll
      for (int i = 0; i < PT; ++i)
#pragma unroll
        for (int j = 0; j < VW; ++j) v[i][j] += u[i][j] * p.y_scale;
    }
  }
  if (p.tokens && p.embed_add) add_embedding();
  if (p.rows == nullptr && (p.tokens || p.y)) {
#pragma unroll
    for (int i = 0; i < PT; ++i) {
      const int c = (tid + i * nt) * VW;
      if (c < p.width) store<VW>(xr + c, v[i]);
    }
  }
  if (p.w_pre) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < PT; ++i)
#pragma unroll
      for (int j = 0; j < VW; ++j) ss = fmaf(v[i][j], v[i][j], ss);
    const float rr = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.eps);
    OutT* o = reinterpret_cast<OutT*>(p.out) + (size_t)r * p.ldo;
#pragma unroll
    for (int i = 0; i < PT; ++i) {
      const int c = (tid + i * nt) * VW;
      if (c < p.width) {
        float w[VW];
#pragma unroll
        for (int j = 0; j < VW; ++j) w[j] = v[i][j] * rr * (p.bias + wa[i][j]);
        store<VW>(o + c, w);
      }
    }
    for (int c = p.width + tid; c < p.ldo; c += nt) o[c] = (OutT)0.f;
  }
}

template <typename OutT, int VW>
int launch_norm(const NormParams& p, int M, cudaStream_t stream) {
  const int groups = (p.width + VW - 1) / VW;
  // one row: as many threads as help its latency; many rows: smaller blocks with a few groups per thread
  const int cap = M <= 64 ? 1024 : 512;
  const int nt = groups >= cap ? (groups > 8 * cap ? 1024 : cap) : ((groups + 31) / 32) * 32;
  const int per = (groups + nt - 1) / nt;
#define PK_NORM_CASE(n)                                                                                \
  if (per <= n) {                                                                                      \
    PK_LAUNCH_PDL((sandwich_norm_kernel<OutT, n, VW>), dim3(M), dim3(nt), (size_t)0, stream, p);       \
    return PK_OK;                                                                                      \
  }
  PK_NORM_CASE(1)
  PK_NORM_CASE(2)
  PK_NORM_CASE(4)
  PK_NORM_CASE(8)
#undef PK_NORM_CASE
  return PK_ERR_UNSUPPORTED;
}

template <typename OutT>
int launch_any(const NormParams& p, int M, cudaStream_t stream) {
  const bool v4 = (p.width & 3) == 0 && ((uintptr_t)p.x & 15) == 0 && (p.y == nullptr || ((p.ldy & 3) == 0 && ((uintptr_t)p.y & 15) == 0)) &&
                  (p.skip == nullptr || ((p.ld_skip & 3) == 0 && ((uintptr_t)p.skip & 15) == 0)) && (p.w_post == nullptr || ((uintptr_t)p.w_post & 15) == 0) &&
                  (p.w_pre == nullptr || (((uintptr_t)p.w_pre & 15) == 0 && (p.ldo & 3) == 0 && ((uintptr_t)p.out & 15) == 0));
  return v4 ? launch_norm<OutT, 4>(p, M, stream) : launch_norm<OutT, 1>(p, M, stream);
}

// ---- per-sequence feedback of greedy decoding: next token and position stay on the device ----

__global__ void feed_tokens_kernel(const int* next, int n, int* tokens, int* pos, int4* seqs, int* hist, int hist_ld, const int* step) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int t = next[i];
  const int s = step[0];
  if (s < hist_ld) hist[(size_t)i * hist_ld + s] = t;
  tokens[i] = t;
  pos[i] += 1;
  seqs[i].w += 1;
}
__global__ void bump_kernel(int* step) { step[0] += 1; }

}  // namespace

// See the head of this file. tokens != null: x is filled from the embedding table (embed_add: the row is added); y != null: the
// (normed) sublayer output x y_scale is added first, skip_w[row] x a row of `skip` being part of it. rows != null: only the M
// listed rows are normed (x stays as it is). width up to 8192 (32768 when a multiple of 4).
PK_API int pk_sandwich_norm(float* x, const int* tokens, const void* embed, int vocab, float embed_scale, int embed_add, const float* y, int ldy,
                            const int* y_rows, int y_top, float y_scale, const void* skip, int ld_skip, int skip_f32, const float* skip_w,
                            const float* w_post, const int* rows, int M, int width, const float* w_pre, int plus_one, float eps, void* out, int ldo, int out_f32, cudaStream_t stream) {
  if (M < 1 || width < 1 || x == nullptr) return PK_ERR_BAD_ARG;
  if (y != nullptr && (ldy < width || (y_rows != nullptr && y_top < 1))) return PK_ERR_BAD_ARG;
  if (skip != nullptr && (y == nullptr || skip_w == nullptr || ld_skip < width)) return PK_ERR_BAD_ARG;
  if (tokens != nullptr && (embed == nullptr || vocab < 1)) return PK_ERR_BAD_ARG;
  if (w_pre != nullptr && (out == nullptr || ldo < width)) return PK_ERR_BAD_ARG;
  NormParams p{x, tokens, (const pk::bf16*)embed, vocab, embed_scale, embed_add, y, ldy, y_rows, y_top, y_scale, skip, skip_w, ld_skip, skip_f32, w_post, rows, width, w_pre,
               plus_one ? 1.f : 0.f, eps, out, ldo};
  return out_f32 ? launch_any<float>(p, M, stream) : launch_any<pk::bf16>(p, M, stream);
}

// next [n] becomes the input token of every row, pos and the
// sequence descriptors' position advance by one, the token is kept in hist[row, step] and step advances.
PK_API int pk_feed_tokens(const int* next, int n, int* tokens, int* pos, void* seqs, int* hist, int hist_ld, int* step, cudaStream_t stream) {
  if (n < 1 || hist_ld < 1) return PK_ERR_BAD_ARG;
  feed_tokens_kernel<<<(n + 127) / 128, 128, 0, stream>>>(next, n, tokens, pos, (int4*)seqs, hist, hist_ld, step);
  PK_CHECK_LAUNCH();
  bump_kernel<<<1, 1, 0, stream>>>(step);
  PK_CHECK_LAUNCH();
  return PK_OK;
}
