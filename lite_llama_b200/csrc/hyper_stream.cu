// Residual kept as several STREAMS x_1 .. x_s (hyper-connections), fp32, [tokens, streams, n].  A sublayer reads a weighted
// sum of the streams and writes all of them at once:
//
//     u = sum_s in[s] x_s;   h = unit_rms(u) * w;   y = sublayer(h)        (optionally y * sigmoid(z + zb) element-wise)
//     x_t <- sum_s mix[s, t] x_s + out[t] y
//
// One pass per sublayer boundary (CTA = token): the finished sublayer's write, the next sublayer's read, its norm, and --
// in steps where every sequence brings one token -- the causal convolution in front of the next sublayer:
//
//   stream_embed   x_1 = .. = x_s = unit_rms(embed[token]) * w0, then the first read
//   stream_mix     write + next read.  y may come as several rows per token (the chosen experts' outputs) and a second
//                  term (a shared expert), summed here in fp32.  With a row list (the output: in = ones, w = the final
//                  norm) only the listed tokens are read and nothing is written back.
//
// The convolution ("input convolution") is hc = h + sum_j cw[:, j] h_(t - taps + 1 + j) on h as stored (rounded to T); a
// slot keeps the last taps - 1 rows of h.  Steps with longer portions run it as a kernel of its own (causal_conv_silu).
#include "common.cuh"
#include "rowvec.cuh"

namespace {

constexpr int kMaxStreams = 8;

struct StreamArgs {
  float* x; int s; int64_t n;                        // streams
  // the finished sublayer: y rows (terms of them per token) + y2, gate logits z + bias zb
  const void* y; int64_t y_stride; int terms; const void* y2; int64_t y2_stride;
  const void* z; int64_t z_stride; const void* zb;
  const float* coef;                                 // [out: s | mix: s x s (from, to)]
  // embedding (stream_embed)
  const int* tokens; const void* embed; const void* embed_w; int64_t vocab;
  // the next read
  const float* in; const void* w; void* h; float eps;
  const int* rows;                                   // listed tokens only, streams not written
  // input convolution of steps of single tokens (taps = 0: none)
  const void* cw; void* tail; void* hc; const int* seq_ctx; const int* seq_slot; int taps;
};

__device__ __forceinline__ float stream_block_sum(float v, float* red) {
  v = warp_reduce_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  t = warp_reduce_sum(t);
  __syncthreads();
  return t;
}

// C consecutive elements (C = 4: one 8- or 16-byte access; 1: scalar)
template <int C, typename T>
__device__ __forceinline__ void load_c(const T* p, float (&v)[C]) {
  if constexpr (C == 4) row_load4(p, v);
  else v[0] = to_f32(p[0]);
}
template <int C, typename T>
__device__ __forceinline__ void store_c(T* p, const float (&v)[C]) {
  if constexpr (C == 4) row_store4(p, v);
  else p[0] = from_f32<T>(v[0]);
}

template <typename T, int S, int C, bool EMBED>      // S = streams (8: up to eight, a.s of them)
__global__ void __launch_bounds__(512) stream_kernel(StreamArgs a) {
  pdl_prologue();
  extern __shared__ __align__(16) float u_row[];     // [n]
  __shared__ float red[32];
  const int ns = S == kMaxStreams ? a.s : S;
  const int64_t o = blockIdx.x, n = a.n;
  const int64_t t = a.rows ? a.rows[o] : o;
  float* xr = a.x + t * ns * n;
  float in[S], out[S], mix[S][S];
#pragma unroll
  for (int i = 0; i < S; ++i) {
    in[i] = i < ns ? a.in[i] : 0.f;
    out[i] = (!EMBED && i < ns) ? a.coef[i] : 0.f;
#pragma unroll
    for (int j = 0; j < S; ++j) mix[i][j] = (!EMBED && i < ns && j < ns) ? a.coef[ns + i * ns + j] : 0.f;
  }
  float ss = 0.f;
  if (EMBED) {
    int64_t tok = a.tokens[t];
    tok = tok < 0 ? 0 : (tok >= a.vocab ? a.vocab - 1 : tok);      // ids are validated on the host; never read outside
    const T* er = (const T*)a.embed + tok * n;
    float se = 0.f, in_sum = 0.f;
    for (int i = 0; i < ns; ++i) in_sum += a.in[i];
    for (int64_t i = threadIdx.x * C; i < n; i += blockDim.x * C) {
      float e[C];
      load_c<C>(er + i, e);
#pragma unroll
      for (int c = 0; c < C; ++c) se = fmaf(e[c], e[c], se);
    }
    const float r = 1.0f / sqrtf(stream_block_sum(se, red) / (float)n + a.eps);
    for (int64_t i = threadIdx.x * C; i < n; i += blockDim.x * C) {
      float e[C], w[C], u[C];
      load_c<C>(er + i, e);
      load_c<C>((const T*)a.embed_w + i, w);
#pragma unroll
      for (int c = 0; c < C; ++c) {
        e[c] = e[c] * r * w[c];
        u[c] = in_sum * e[c];
        ss = fmaf(u[c], u[c], ss);
        u_row[i + c] = u[c];
      }
      for (int j = 0; j < ns; ++j) store_c<C>(xr + j * n + i, e);
    }
  } else {
    const T* yr = (const T*)a.y + t * a.terms * a.y_stride;
    const T* y2 = a.y2 ? (const T*)a.y2 + t * a.y2_stride : nullptr;
    const T* zr = a.z ? (const T*)a.z + t * a.z_stride : nullptr;
    for (int64_t i = threadIdx.x * C; i < n; i += blockDim.x * C) {
      float x[S][C], y[C];
#pragma unroll
      for (int j = 0; j < S; ++j)
        if (j < ns) load_c<C>(xr + j * n + i, x[j]);
      load_c<C>(yr + i, y);
      for (int k = 1; k < a.terms; ++k) {
        float v[C];
        load_c<C>(yr + k * a.y_stride + i, v);
#pragma unroll
        for (int c = 0; c < C; ++c) y[c] += v[c];
      }
      if (y2) {
        float v[C];
        load_c<C>(y2 + i, v);
#pragma unroll
        for (int c = 0; c < C; ++c) y[c] += v[c];
      }
      if (zr) {
        float z[C], b[C];
        load_c<C>(zr + i, z);
        load_c<C>((const T*)a.zb + i, b);
#pragma unroll
        for (int c = 0; c < C; ++c) y[c] /= 1.0f + expf(-(z[c] + b[c]));
      }
      float u[C];
#pragma unroll
      for (int c = 0; c < C; ++c) u[c] = 0.f;
#pragma unroll
      for (int j = 0; j < S; ++j) {
        if (j >= ns) continue;
        float v[C];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          v[c] = out[j] * y[c];
#pragma unroll
          for (int k = 0; k < S; ++k)
            if (k < ns) v[c] = fmaf(mix[k][j], x[k][c], v[c]);
          u[c] = fmaf(in[j], v[c], u[c]);
        }
        if (!a.rows) store_c<C>(xr + j * n + i, v);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) { ss = fmaf(u[c], u[c], ss); u_row[i + c] = u[c]; }
    }
  }
  const float rstd = 1.0f / sqrtf(stream_block_sum(ss, red) / (float)n + a.eps);
  T* hr = (T*)a.h + o * n;
  const int keep = a.taps - 1;
  const int ctx = a.taps > 0 ? a.seq_ctx[t] : 0;      // single-token step: token t is sequence t
  T* tail = a.taps > 1 ? (T*)a.tail + (int64_t)a.seq_slot[t] * keep * n : nullptr;
  for (int64_t i = threadIdx.x * C; i < n; i += blockDim.x * C) {
    float w[C], h[C];
    load_c<C>((const T*)a.w + i, w);
#pragma unroll
    for (int c = 0; c < C; ++c) h[c] = to_f32(from_f32<T>(u_row[i + c] * rstd * w[c]));
    store_c<C>(hr + i, h);
    if (a.taps > 0) {
      const T* cw = (const T*)a.cw + i * a.taps;
      float acc[C];
#pragma unroll
      for (int c = 0; c < C; ++c) acc[c] = fmaf(to_f32(cw[c * a.taps + keep]), h[c], h[c]);
      // tail row j holds the input keep - j tokens back; newest first, the order of causal_conv_silu
      for (int j = keep - 1; j >= 0; --j) {
        float v[C];
#pragma unroll
        for (int c = 0; c < C; ++c) v[c] = 0.f;
        if (ctx - keep + j >= 0) load_c<C>(tail + (int64_t)j * n + i, v);
#pragma unroll
        for (int c = 0; c < C; ++c) acc[c] = fmaf(to_f32(cw[c * a.taps + j]), v[c], acc[c]);
      }
      for (int j = 0; j < keep - 1; ++j) {
        float v[C];
#pragma unroll
        for (int c = 0; c < C; ++c) v[c] = 0.f;
        if (ctx - keep + j + 1 >= 0) load_c<C>(tail + (int64_t)(j + 1) * n + i, v);
        store_c<C>(tail + (int64_t)j * n + i, v);
      }
      if (keep > 0) store_c<C>(tail + (int64_t)(keep - 1) * n + i, h);
      store_c<C>((T*)a.hc + o * n + i, acc);
    }
  }
}

template <typename T, int C, bool EMBED>
int launch_stream(const StreamArgs& a, int64_t tokens, cudaStream_t st) {
  const int64_t per = cdiv64(a.n, C);
  const int64_t most = tokens <= 2 * b2l_num_sms() ? 512 : 256;        // few tokens: the latency of one row is all there is
  const int threads = per >= most ? (int)most : (int)(cdiv64(per, 32) * 32);
  const size_t smem = (size_t)a.n * sizeof(float);
  B2L_REQUIRE((int64_t)smem <= b2l_max_smem_optin() - 1024, "stream kernels: rows of %lld elements", (long long)a.n);
#define B2L_STREAM(S)                                                                                     \
  do {                                                                                                    \
    static int cache[64] = {0};                                                                           \
    if (smem > 40 * 1024) B2L_CUDA_CHECK(b2l_ensure_dynamic_smem(stream_kernel<T, S, C, EMBED>, (int)smem, cache)); \
    b2l_launch(stream_kernel<T, S, C, EMBED>, dim3((unsigned)tokens), dim3(threads), smem, st, a);        \
  } while (0)
  switch (a.s) {
    case 1: B2L_STREAM(1); break;
    case 2: B2L_STREAM(2); break;
    case 3: B2L_STREAM(3); break;
    case 4: B2L_STREAM(4); break;
    default: B2L_STREAM(kMaxStreams);
  }
#undef B2L_STREAM
  B2L_LAUNCH_CHECK();
  return B2L_OK;
}

}  // namespace

/* The read of a sublayer: in_f32 [streams], weight [n], h [tokens, n] in dtype; with taps > 0 (every token of the step is
 * a sequence of its own) also hc = h + its causal convolution: conv_w [n, taps], tail [slots, taps - 1, n] advanced. */
extern "C" int b2l_stream_embed(void* streams_f32, const void* tokens_i32, const void* embed, const void* embed_weight,
                                int64_t vocab, const void* in_f32, const void* weight, void* h, const void* conv_w,
                                void* tail, void* hc, const void* seq_ctx, const void* seq_slot, int taps, int64_t tokens,
                                int streams, int64_t n, float eps, int dtype, void* stream) {
  B2L_REQUIRE(streams_f32 && tokens_i32 && embed && embed_weight && in_f32 && weight && h, "stream_embed: null pointer");
  B2L_REQUIRE(streams >= 1 && streams <= kMaxStreams && n > 0 && vocab > 0 && taps >= 0, "stream_embed: %d streams of %lld",
              streams, (long long)n);
  B2L_REQUIRE(taps == 0 || (conv_w && hc && seq_ctx && seq_slot && (tail || taps == 1)), "stream_embed: null convolution pointer");
  if (tokens <= 0) return B2L_OK;
  StreamArgs a = {};
  a.x = (float*)streams_f32; a.s = streams; a.n = n;
  a.tokens = (const int*)tokens_i32; a.embed = embed; a.embed_w = embed_weight; a.vocab = vocab;
  a.in = (const float*)in_f32; a.w = weight; a.h = h; a.eps = eps;
  a.cw = conv_w; a.tail = tail; a.hc = hc; a.seq_ctx = (const int*)seq_ctx; a.seq_slot = (const int*)seq_slot; a.taps = taps;
  int rc = B2L_OK;
  B2L_DISPATCH_FLOAT(dtype, "stream_embed", {
    const bool v4 = n % 4 == 0 && (uintptr_t)streams_f32 % 16 == 0 && row_aligned4<T>(embed) && row_aligned4<T>(embed_weight) &&
                    row_aligned4<T>(weight) && row_aligned4<T>(h) && row_aligned4<T>(tail) && row_aligned4<T>(hc);
    rc = v4 ? launch_stream<T, 4, true>(a, tokens, (cudaStream_t)stream) : launch_stream<T, 1, true>(a, tokens, (cudaStream_t)stream);
  });
  return rc;
}

/* The write of a sublayer and the next read.  y: `terms` rows per token (row stride given), y2 (nullable) one more; z
 * (nullable): the sum times sigmoid(z + z_bias).  coef_f32 = [out: streams | mix: streams x streams (from, to)].
 * rows_i32 (nullable, `tokens` entries): only these tokens, h compact, the streams stay as they are. */
extern "C" int b2l_stream_mix(void* streams_f32, const void* y, int64_t y_row_stride, int terms, const void* y2,
                              int64_t y2_row_stride, const void* z, int64_t z_row_stride, const void* z_bias,
                              const void* coef_f32, const void* in_f32, const void* weight, void* h, const void* rows_i32,
                              const void* conv_w, void* tail, void* hc, const void* seq_ctx, const void* seq_slot,
                              int taps, int64_t tokens, int streams, int64_t n, float eps, int dtype, void* stream) {
  B2L_REQUIRE(streams_f32 && y && coef_f32 && in_f32 && weight && h && (!z || z_bias), "stream_mix: null pointer");
  B2L_REQUIRE(streams >= 1 && streams <= kMaxStreams && n > 0 && terms >= 1 && taps >= 0, "stream_mix: %d streams of %lld, %d terms",
              streams, (long long)n, terms);
  B2L_REQUIRE(taps == 0 || (!rows_i32 && conv_w && hc && seq_ctx && seq_slot && (tail || taps == 1)),
              "stream_mix: null convolution pointer");
  if (tokens <= 0) return B2L_OK;
  StreamArgs a = {};
  a.x = (float*)streams_f32; a.s = streams; a.n = n;
  a.y = y; a.y_stride = y_row_stride; a.terms = terms; a.y2 = y2; a.y2_stride = y2_row_stride;
  a.z = z; a.z_stride = z_row_stride; a.zb = z_bias; a.coef = (const float*)coef_f32;
  a.in = (const float*)in_f32; a.w = weight; a.h = h; a.eps = eps; a.rows = (const int*)rows_i32;
  a.cw = conv_w; a.tail = tail; a.hc = hc; a.seq_ctx = (const int*)seq_ctx; a.seq_slot = (const int*)seq_slot; a.taps = taps;
  int rc = B2L_OK;
  B2L_DISPATCH_FLOAT(dtype, "stream_mix", {
    const bool v4 = n % 4 == 0 && (uintptr_t)streams_f32 % 16 == 0 && y_row_stride % 4 == 0 && y2_row_stride % 4 == 0 &&
                    z_row_stride % 4 == 0 && row_aligned4<T>(y) && row_aligned4<T>(y2) && row_aligned4<T>(z) &&
                    row_aligned4<T>(z_bias) && row_aligned4<T>(weight) && row_aligned4<T>(h) && row_aligned4<T>(tail) &&
                    row_aligned4<T>(hc);
    rc = v4 ? launch_stream<T, 4, false>(a, tokens, (cudaStream_t)stream) : launch_stream<T, 1, false>(a, tokens, (cudaStream_t)stream);
  });
  return rc;
}
