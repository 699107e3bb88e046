// Residual of designs whose sublayers read an ELEMENT-WISE norm of it, h = tanh(alpha v) * w + b, and add their result as
// it is (no output norm).  Nothing in a row depends on the rest of the row, so one pass per sublayer boundary does all of
// it without a reduction, spread over the grid by elements whatever the number of tokens:
//
//     v = residual + y                         the finished sublayer (or, `first`: v starts at 0)
//       + addend                               a second term of it (a shared expert)
//       + embed_scale * embed[token]           where a run of looped layers starts again (recomputed from the table: no copy
//                                              of the embedding output is kept); with `first` this IS the embedding
//       + step                                 a vector that marks the pass of a loop
//     residual = v;   act = tanh(alpha v) * w + b
//
// y may come as the weighted outputs of a token's chosen experts, [tokens, top, n], summed here in fp32.  Expert ids from
// `experts` on are identity experts: they have no rows in y, their output is their input x times the weight.
// With a row list (the output norm) only the listed tokens are read and the residual is not written.
#include "common.cuh"

namespace {

struct TanhStreamArgs {
  float* residual; void* act;
  const void* y; int64_t y_stride; int top;
  const int* ids; const float* weights; int experts; const void* x; int64_t x_stride;
  const void* addend;
  const int* tokens; const void* embed; int64_t vocab; float embed_scale;
  const void* step; int first;
  const void* alpha; const void* w; const void* b;
  const int* rows; int64_t chunks, total;        // chunks of C elements per row; chunks of all rows
};

// C consecutive elements: 16-byte accesses of T (C = 8 for the 16-bit types, 4 for fp32; the fp32 residual then takes two
// or one), or scalars (C = 1)
template <int C, typename T>
__device__ __forceinline__ void load_c(const T* p, float (&v)[C]) {
  if constexpr (C == 1) {
    v[0] = to_f32(p[0]);
  } else {
    constexpr int V = 16 / (int)sizeof(T);
#pragma unroll
    for (int i = 0; i < C; i += V) {
      const uint4 raw = *reinterpret_cast<const uint4*>(p + i);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int c = 0; c < V; ++c) v[i + c] = to_f32(e[c]);
    }
  }
}
template <int C, typename T>
__device__ __forceinline__ void store_c(T* p, const float (&v)[C]) {
  if constexpr (C == 1) {
    p[0] = from_f32<T>(v[0]);
  } else {
    constexpr int V = 16 / (int)sizeof(T);
#pragma unroll
    for (int i = 0; i < C; i += V) {
      uint4 raw;
      T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
      for (int c = 0; c < V; ++c) e[c] = from_f32<T>(v[i + c]);
      *reinterpret_cast<uint4*>(p + i) = raw;
    }
  }
}
template <int C, typename T>
__device__ __forceinline__ void add_c(const T* p, float scale, float (&v)[C]) {
  float e[C];
  load_c<C>(p, e);
#pragma unroll
  for (int c = 0; c < C; ++c) v[c] = fmaf(e[c], scale, v[c]);
}

template <typename T, int C>
__global__ void __launch_bounds__(256) tanh_norm_stream_kernel(TanhStreamArgs a) {
  pdl_prologue();
  const int64_t idx = (int64_t)blockIdx.x * 256 + threadIdx.x;
  if (idx >= a.total) return;
  const int64_t o = idx / a.chunks, i = (idx - o * a.chunks) * C, n = a.chunks * C;
  const int64_t t = a.rows ? a.rows[o] : o;
  float v[C];
  if (a.first) {
#pragma unroll
    for (int c = 0; c < C; ++c) v[c] = 0.f;
  } else {
    load_c<C>(a.residual + t * n + i, v);
  }
  if (a.y) {
    if (a.top == 0) {
      add_c<C>((const T*)a.y + t * a.y_stride + i, 1.0f, v);
    } else {
      constexpr int B = 4;                       // rows in flight
      float sum[C];
#pragma unroll
      for (int c = 0; c < C; ++c) sum[c] = 0.f;
      for (int k0 = 0; k0 < a.top; k0 += B) {
        float e[B][C], f[B];
#pragma unroll
        for (int u = 0; u < B; ++u) {
          f[u] = 0.f;
          if (k0 + u >= a.top) continue;
          const int64_t slot = t * a.top + k0 + u;
          const bool expert = a.ids[slot] < a.experts;
          f[u] = expert ? 1.0f : a.weights[slot];
          load_c<C>(expert ? (const T*)a.y + slot * a.y_stride + i : (const T*)a.x + t * a.x_stride + i, e[u]);
        }
#pragma unroll
        for (int u = 0; u < B; ++u) {
          if (k0 + u >= a.top) continue;
#pragma unroll
          for (int c = 0; c < C; ++c) sum[c] = fmaf(e[u][c], f[u], sum[c]);
        }
      }
      if (a.addend) add_c<C>((const T*)a.addend + t * n + i, 1.0f, sum);
#pragma unroll
      for (int c = 0; c < C; ++c) v[c] += sum[c];
    }
  }
  if (a.tokens) {
    int64_t tok = a.tokens[t];
    tok = tok < 0 ? 0 : (tok >= a.vocab ? a.vocab - 1 : tok);      // ids are validated on the host; never read outside
    float e[C];
    load_c<C>((const T*)a.embed + tok * n + i, e);
#pragma unroll
    for (int c = 0; c < C; ++c) v[c] += e[c] * a.embed_scale;
  }
  if (a.step) add_c<C>((const T*)a.step + i, 1.0f, v);
  if (!a.rows) store_c<C>(a.residual + t * n + i, v);
  if (!a.act) return;
  const float alpha = to_f32(*(const T*)a.alpha);
  float w[C], b[C];
  load_c<C>((const T*)a.w + i, w);
  load_c<C>((const T*)a.b + i, b);
#pragma unroll
  for (int c = 0; c < C; ++c) v[c] = fmaf(tanhf(alpha * v[c]), w[c], b[c]);
  store_c<C>((T*)a.act + o * n + i, v);
}

}  // namespace

extern "C" int b2l_tanh_norm_stream(void* residual_f32, void* act, const void* y, int64_t y_row_stride, int top,
                                    const void* ids_i32, const void* weights_f32, int experts, const void* x,
                                    int64_t x_row_stride, const void* addend, const void* tokens_i32, const void* embed,
                                    int64_t vocab, float embed_scale, const void* step, int first, const void* alpha,
                                    const void* w, const void* b, const void* rows_i32, int64_t num_rows, int64_t n,
                                    int dtype, void* stream) {
  B2L_REQUIRE(residual_f32 && n > 0 && num_rows >= 0 && top >= 0, "tanh_norm_stream: bad shape");
  B2L_REQUIRE(!act || (alpha && w && b), "tanh_norm_stream: a norm needs its weight, shift and alpha");
  B2L_REQUIRE(top == 0 || (y && ids_i32 && weights_f32 && x), "tanh_norm_stream: expert terms need ids, weights and their input");
  B2L_REQUIRE(!addend || top > 0, "tanh_norm_stream: a second term joins expert terms");
  B2L_REQUIRE(!tokens_i32 || (embed && vocab > 0), "tanh_norm_stream: no embedding table");
  B2L_REQUIRE(!first || (!y && !rows_i32), "tanh_norm_stream: the first call has no sublayer to add");
  if (num_rows == 0) return B2L_OK;
  cudaStream_t st = (cudaStream_t)stream;
  TanhStreamArgs a = {};
  a.residual = (float*)residual_f32; a.act = act; a.y = y; a.y_stride = y_row_stride; a.top = top;
  a.ids = (const int*)ids_i32; a.weights = (const float*)weights_f32; a.experts = experts; a.x = x; a.x_stride = x_row_stride;
  a.addend = addend; a.tokens = (const int*)tokens_i32; a.embed = embed; a.vocab = vocab; a.embed_scale = embed_scale;
  a.step = step; a.first = first; a.alpha = alpha; a.w = w; a.b = b; a.rows = (const int*)rows_i32;
  B2L_DISPATCH_FLOAT(dtype, "tanh_norm_stream", {
    constexpr int C = 16 / (int)sizeof(T);
    auto al = [](const void* p) { return (uintptr_t)p % 16 == 0; };             // true for absent operands too
    const bool vec = n % C == 0 && (!y || y_row_stride % C == 0) && (!x || x_row_stride % C == 0) && al(residual_f32) &&
                     al(act) && al(y) && al(x) && al(addend) && al(embed) && al(step) && al(w) && al(b);
    a.chunks = vec ? n / C : n;
    a.total = a.chunks * num_rows;
    const dim3 grid((unsigned)cdiv64(a.total, 256));
    if (vec) b2l_launch(tanh_norm_stream_kernel<T, C>, grid, dim3(256), (size_t)0, st, a);
    else b2l_launch(tanh_norm_stream_kernel<T, 1>, grid, dim3(256), (size_t)0, st, a);
  });
  B2L_LAUNCH_CHECK();
  return B2L_OK;
}
