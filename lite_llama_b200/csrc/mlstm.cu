// Matrix memory with exponential gates (mLSTM) over RAGGED steps.  Per head a memory S [D x V], a normaliser n [D] and a
// running log scale m, all fp32, kept per request slot as [S | n | m] (padded to a multiple of 4 floats):
//
//     i = cap tanh((zi + bi) / cap),   f = logsigmoid(cap tanh((zf + bf) / cap))            one number per head
//     m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n likewise with k alone;  m <- m'
//     y = S^T q / (max(|n . q|, e^(-m)) + 1e-6),        q = q_scale * (projection column)
//
// A sequence without cached tokens starts from S = n = m = 0 and never reads its slot.
//
//   mlstm_scan    token by token, any dtype and size: CTA = (64 value columns, head, sequence), a thread keeps 4 columns of
//                 D / 16 memory rows in registers and its rows of n.  Serves single tokens, fp32 and odd shapes.
//   mlstm_chunk   prompt portions in chunks of 64 tokens on mma.sync tiles (16-bit activations).  With F the running sum
//                 of f inside the chunk, a_j = i_j - F_j and M_i = max(m, a_0 .. a_i) the recurrence unrolls to
//                     m_i = F_i + M_i
//                     S_i = e^(m - M_i) S + sum_{j <= i} e^(a_j - M_i) k_j v_j^T        (every exponent <= 0)
//                 so a chunk is the products  A = Q K^T,  W = e^(a_j - M_i) A (j <= i),  Y = W V + e^(m - M_i) Q S  and
//                 S <- e^(m - M_last) S + K^T (e^(a_j - M_last) V);  the denominators are the row sums of W plus
//                 e^(m - M_i) Q n.  Every fp32 factor that enters a product (W, S, the scaled V) goes in as the sum of two
//                 16-bit halves, so nothing but q, k, v themselves (16-bit already) is rounded; sums, memory, gates and
//                 normaliser stay fp32.
// Column tiles of one head each form the head's n and m for themselves; the tile that finishes last (a ticket per head and
// sequence, left at zero) stores them, when every other tile has long read the old ones.
#include "common.cuh"

namespace {

struct MlstmArgs {
  float* y; float* state; int64_t head_floats;      // floats of one head's [S | n | m] block
  const void* q; int64_t q_stride; const void* k; int64_t k_stride; const void* v; int64_t v_stride;
  const void* zi; int64_t zi_stride; const void* zf; int64_t zf_stride; const void* bi; const void* bf;
  const int* seq_start; const int* seq_ctx; const int* seq_slot; const int* seq_list;
  int* tickets;
  int H, D, V;
  float q_scale, cap;
};

__device__ __forceinline__ float log_sigmoid(float x) {
  return x >= 0.f ? -log1pf(expf(-x)) : x - log1pf(expf(x));
}
__device__ __forceinline__ float soft_bound(float z, float cap) { return cap > 0.f ? cap * tanhf(z / cap) : z; }

// true in every thread of the CTA that is the last of `tiles` to get here (the others' reads are done)
__device__ __forceinline__ bool last_tile(int* ticket, int tiles, int* flag) {
  if (tiles == 1) return true;
  __syncthreads();
  if (threadIdx.x == 0) {
    const int t = atomicAdd(ticket, 1);
    *flag = t == tiles - 1;
    if (t == tiles - 1) *ticket = 0;
  }
  __syncthreads();
  return *flag != 0;
}

// ---- token by token -------------------------------------------------------------------------------------------------
constexpr int kScanCols = 64, kScanThreads = 256, kScanTok = 8;

template <typename T, int R>                        // R = memory rows per thread: row r = group + 16 * j, D <= 16 R
__global__ void __launch_bounds__(kScanThreads) mlstm_scan_kernel(MlstmArgs a) {
  pdl_prologue();
  __shared__ float qs[kScanTok][16 * R], ks[kScanTok][16 * R];
  __shared__ float vs[kScanTok][kScanCols];
  __shared__ float gs[kScanTok][2];
  __shared__ float red[kScanThreads / 32][kScanCols + 1];
  __shared__ int flag;
  const int D = a.D, V = a.V, H = a.H, h = blockIdx.y;
  const int s = a.seq_list ? a.seq_list[blockIdx.z] : blockIdx.z;
  const int start = a.seq_start[s], len = a.seq_start[s + 1] - start, ctx = a.seq_ctx[s];
  if (len <= 0) return;
  float* st = a.state + ((int64_t)a.seq_slot[s] * H + h) * a.head_floats;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int cg = tid & 15, rg = tid >> 4;           // column group (4 columns), row group
  const int c0 = blockIdx.x * kScanCols, col = c0 + cg * 4;
  const bool vec = V % 4 == 0;                      // head blocks and rows start on 16 bytes
  float S[R][4], n[R], m = 0.f;
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int d = rg + 16 * j;
    S[j][0] = S[j][1] = S[j][2] = S[j][3] = n[j] = 0.f;
    if (ctx > 0 && d < D) {
      n[j] = st[(int64_t)D * V + d];
      const float* p = st + (int64_t)d * V + col;
      if (vec) {
        if (col < V) { const float4 r = *reinterpret_cast<const float4*>(p); S[j][0] = r.x; S[j][1] = r.y; S[j][2] = r.z; S[j][3] = r.w; }
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) if (col + e < V) S[j][e] = p[e];
      }
    }
  }
  if (ctx > 0) m = st[(int64_t)D * V + D];
  const T* q = (const T*)a.q + (int64_t)h * D;
  const T* k = (const T*)a.k + (int64_t)h * D;
  const T* v = (const T*)a.v + (int64_t)h * V;
  const float bi = to_f32(((const T*)a.bi)[h]), bf = to_f32(((const T*)a.bf)[h]);
  for (int t0 = 0; t0 < len; t0 += kScanTok) {
    const int nt = min(kScanTok, len - t0);
    __syncthreads();
    for (int i = tid; i < nt * 16 * R; i += kScanThreads) {
      const int t = i / (16 * R), d = i - t * (16 * R);
      const int64_t row = start + t0 + t;
      qs[t][d] = d < D ? to_f32(q[row * a.q_stride + d]) * a.q_scale : 0.f;
      ks[t][d] = d < D ? to_f32(k[row * a.k_stride + d]) : 0.f;
    }
    for (int i = tid; i < nt * kScanCols; i += kScanThreads) {
      const int t = i / kScanCols, c = i - t * kScanCols;
      vs[t][c] = c0 + c < V ? to_f32(v[(int64_t)(start + t0 + t) * a.v_stride + c0 + c]) : 0.f;
    }
    if (tid < nt) {
      const int64_t row = start + t0 + tid;
      gs[tid][0] = soft_bound(to_f32(((const T*)a.zi)[row * a.zi_stride + h]) + bi, a.cap);
      gs[tid][1] = log_sigmoid(soft_bound(to_f32(((const T*)a.zf)[row * a.zf_stride + h]) + bf, a.cap));
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float gi = gs[t][0], fm = gs[t][1] + m, mn = fmaxf(fm, gi);
      const float keep = expf(fm - mn), write = expf(gi - mn);
      m = mn;
      float o[4] = {0.f, 0.f, 0.f, 0.f}, nq = 0.f;
      const float v0 = vs[t][cg * 4], v1 = vs[t][cg * 4 + 1], v2 = vs[t][cg * 4 + 2], v3 = vs[t][cg * 4 + 3];
#pragma unroll
      for (int j = 0; j < R; ++j) {
        const float wk = write * ks[t][rg + 16 * j], qq = qs[t][rg + 16 * j];
        S[j][0] = fmaf(keep, S[j][0], wk * v0); S[j][1] = fmaf(keep, S[j][1], wk * v1);
        S[j][2] = fmaf(keep, S[j][2], wk * v2); S[j][3] = fmaf(keep, S[j][3], wk * v3);
        n[j] = fmaf(keep, n[j], wk);
        o[0] = fmaf(S[j][0], qq, o[0]); o[1] = fmaf(S[j][1], qq, o[1]);
        o[2] = fmaf(S[j][2], qq, o[2]); o[3] = fmaf(S[j][3], qq, o[3]);
        nq = fmaf(n[j], qq, nq);
      }
      // the two row groups of a warp, then the eight warps (in order)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
      nq += __shfl_xor_sync(0xffffffffu, nq, 16);
      if (lane < 16) {
#pragma unroll
        for (int e = 0; e < 4; ++e) red[warp][cg * 4 + e] = o[e];
        if (lane == 0) red[warp][kScanCols] = nq;
      }
      __syncthreads();
      if (tid < kScanCols && c0 + tid < V) {
        float num = 0.f, den = 0.f;
#pragma unroll
        for (int w = 0; w < kScanThreads / 32; ++w) { num += red[w][tid]; den += red[w][kScanCols]; }
        a.y[(int64_t)(start + t0 + t) * H * V + (int64_t)h * V + c0 + tid] = num / (fmaxf(fabsf(den), expf(-m)) + 1e-6f);
      }
      __syncthreads();
    }
  }
#pragma unroll
  for (int j = 0; j < R; ++j) {
    const int d = rg + 16 * j;
    if (d >= D) continue;
    float* p = st + (int64_t)d * V + col;
    if (vec) {
      if (col < V) *reinterpret_cast<float4*>(p) = make_float4(S[j][0], S[j][1], S[j][2], S[j][3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) if (col + e < V) p[e] = S[j][e];
    }
  }
  if (last_tile(a.tickets + blockIdx.z * H + h, gridDim.x, &flag) && cg == 0) {
#pragma unroll
    for (int j = 0; j < R; ++j) {
      const int d = rg + 16 * j;
      if (d < D) st[(int64_t)D * V + d] = n[j];
    }
    if (tid == 0) st[(int64_t)D * V + D] = m;
  }
}

// ---- chunks on the tensor cores -------------------------------------------------------------------------------------
constexpr int kC = 64, kChunkThreads = 128;
constexpr float kL2e = 1.4426950408889634f;

// (x, y) as two packed 16-bit pairs whose sum is (x, y) to ~16 mantissa bits
template <typename T>
__device__ __forceinline__ void halves2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const T hx = from_f32<T>(x), hy = from_f32<T>(y);
  hi = pack2<T>(to_f32(hx), to_f32(hy));
  lo = pack2<T>(x - to_f32(hx), y - to_f32(hy));
}

// 8 elements from p, the first `valid` of them (0 beyond)
template <typename T>
__device__ __forceinline__ uint4 load8(const T* p, int valid, bool vec) {
  uint4 r = make_uint4(0u, 0u, 0u, 0u);
  if (vec && valid >= 8) return ldg_128(p);
  T* e = reinterpret_cast<T*>(&r);
#pragma unroll
  for (int i = 0; i < 8; ++i) if (i < valid) e[i] = p[i];
  return r;
}

template <typename T, int N, int P>                 // D <= N, a tile of P value columns
__global__ void __launch_bounds__(kChunkThreads) mlstm_chunk_kernel(MlstmArgs a, int vec) {
  pdl_prologue();
  extern __shared__ __align__(16) uint8_t mc_smem[];
  constexpr int QP = (N + 8) * 2, VP = (P + 8) * 2;           // row pitches in bytes (16-bit tiles)
  constexpr int SP = P + 4;                                    // fp32 memory pitch in floats
  uint8_t* sQ = mc_smem;                                       // [kC][N + 8]
  uint8_t* sK = sQ + kC * QP;
  uint8_t* sV = sK + kC * QP;                                  // [kC][P + 8]
  uint8_t* sVh = sV + kC * VP;                                 // e^(a_j - M_last) v: high halves
  uint8_t* sVl = sVh + kC * VP;                                // low halves
  float* sS = reinterpret_cast<float*>(sVl + kC * VP);         // [N][SP]
  float* sN = sS + N * SP;                                     // [N]
  float* sA = sN + N;                                          // [kC] a_j log2(e)
  float* sM = sA + kC;                                         // [kC] M_i log2(e)
  float* sCar = sM + kC;                                       // [kC] q_scale e^(m - M_i)
  float* sFloor = sCar + kC;                                   // [kC] e^(-m_i)
  float* sW = sFloor + kC;                                     // [kC] e^(a_j - M_last), 0 past the end
  float* sScal = sW + kC;                                      // [2] e^(m - M_last), new m
  __shared__ int flag;
  const int h = blockIdx.x, H = a.H, D = a.D, V = a.V, p0 = blockIdx.z * P;
  const int s = a.seq_list ? a.seq_list[blockIdx.y] : blockIdx.y;
  const int start = a.seq_start[s], len = a.seq_start[s + 1] - start, ctx = a.seq_ctx[s];
  if (len <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int gq = lane >> 2, tq = lane & 3;
  const int pc = min(P, V - p0);                               // live columns of the tile
  float* st = a.state + ((int64_t)a.seq_slot[s] * H + h) * a.head_floats;
  for (int i = tid; i < N * P; i += kChunkThreads) {
    const int d = i / P, p = i - d * P;
    sS[d * SP + p] = (ctx > 0 && d < D && p < pc) ? st[(int64_t)d * V + p0 + p] : 0.f;
  }
  for (int d = tid; d < N; d += kChunkThreads) sN[d] = (ctx > 0 && d < D) ? st[(int64_t)D * V + d] : 0.f;
  float m = ctx > 0 ? st[(int64_t)D * V + D] : 0.f;            // carried scale (every thread)
  const T* qg = (const T*)a.q + (int64_t)h * D;
  const T* kg = (const T*)a.k + (int64_t)h * D;
  const T* vg = (const T*)a.v + (int64_t)h * V + p0;
  const float bi = to_f32(((const T*)a.bi)[h]), bf = to_f32(((const T*)a.bf)[h]);
  bool carried = ctx > 0;
  // a chunk's rows travel global -> registers -> shared memory; the NEXT chunk's loads are issued before the products
  // of the current one and land while they run
  constexpr int QV = kC * (N / 8) / kChunkThreads, VV = kC * (P / 8) / kChunkThreads;
  uint4 pq[QV], pk[QV], pv[VV];
  float zi[2], zf[2];                                          // warp 0: gate logits of tokens 2 lane, 2 lane + 1
  auto fetch = [&](int cs) {
    const int cnt = min(kC, len - cs);
#pragma unroll
    for (int u = 0; u < QV; ++u) {
      const int i = tid + u * kChunkThreads, j = i / (N / 8), c = (i - j * (N / 8)) * 8;
      const int64_t row = start + cs + j;
      const int valid = j < cnt ? D - c : 0;
      pq[u] = load8(qg + row * a.q_stride + c, valid, vec);
      pk[u] = load8(kg + row * a.k_stride + c, valid, vec);
    }
#pragma unroll
    for (int u = 0; u < VV; ++u) {
      const int i = tid + u * kChunkThreads, j = i / (P / 8), c = (i - j * (P / 8)) * 8;
      pv[u] = load8(vg + (int64_t)(start + cs + j) * a.v_stride + c, j < cnt ? pc - c : 0, vec);
    }
    if (warp == 0) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = 2 * lane + e;
        const int64_t row = start + cs + j;
        zi[e] = j < cnt ? to_f32(((const T*)a.zi)[row * a.zi_stride + h]) : 0.f;
        zf[e] = j < cnt ? to_f32(((const T*)a.zf)[row * a.zf_stride + h]) : 0.f;
      }
    }
  };
  // warp 0: gates, their running sums and maxima, and every weight of the chunk that depends on one token
  auto gates = [&](int cnt) {
    float f[2], g[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const bool in = 2 * lane + e < cnt;
      f[e] = in ? log_sigmoid(soft_bound(zf[e] + bf, a.cap)) : 0.f;
      g[e] = in ? soft_bound(zi[e] + bi, a.cap) : -INFINITY;
    }
    float run = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += x;
    }
    const float F1 = run, F0 = run - f[1];                     // running sums at tokens 2 lane, 2 lane + 1
    const float A0 = g[0] - F0, A1 = g[1] - F1;
    float mx = fmaxf(A0, A1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float x = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, x);
    }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);
    before = lane == 0 ? m : fmaxf(m, before);
    const float M0 = fmaxf(before, A0), M1 = fmaxf(M0, A1);
    const float Mlast = __shfl_sync(0xffffffffu, M1, 31), Flast = __shfl_sync(0xffffffffu, F1, 31);   // tokens past the end add nothing
    const int j = 2 * lane;
    sA[j] = A0 * kL2e; sA[j + 1] = A1 * kL2e;
    sM[j] = M0 * kL2e; sM[j + 1] = M1 * kL2e;
    sCar[j] = a.q_scale * expf(m - M0); sCar[j + 1] = a.q_scale * expf(m - M1);
    sFloor[j] = expf(-(F0 + M0)); sFloor[j + 1] = expf(-(F1 + M1));
    sW[j] = expf(A0 - Mlast); sW[j + 1] = expf(A1 - Mlast);     // exp(-inf) = 0 past the end
    if (lane == 0) { sScal[0] = expf(m - Mlast); sScal[1] = Flast + Mlast; }
  };
  auto commit = [&]() {
#pragma unroll
    for (int u = 0; u < QV; ++u) {
      const int i = tid + u * kChunkThreads, j = i / (N / 8), c = (i - j * (N / 8)) * 8;
      *reinterpret_cast<uint4*>(sQ + j * QP + c * 2) = pq[u];
      *reinterpret_cast<uint4*>(sK + j * QP + c * 2) = pk[u];
    }
#pragma unroll
    for (int u = 0; u < VV; ++u) {
      const int i = tid + u * kChunkThreads, j = i / (P / 8), c = (i - j * (P / 8)) * 8;
      const float w = sW[j];
      const T* ev = reinterpret_cast<const T*>(&pv[u]);
      uint4 rh, rl;
      T* oh = reinterpret_cast<T*>(&rh);
      T* ol = reinterpret_cast<T*>(&rl);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float x = to_f32(ev[e]) * w;
        oh[e] = from_f32<T>(x);
        ol[e] = from_f32<T>(x - to_f32(oh[e]));
      }
      *reinterpret_cast<uint4*>(sV + j * VP + c * 2) = pv[u];
      *reinterpret_cast<uint4*>(sVh + j * VP + c * 2) = rh;
      *reinterpret_cast<uint4*>(sVl + j * VP + c * 2) = rl;
    }
  };
  fetch(0);
  for (int cs = 0; cs < len; cs += kC) {
    const int cnt = min(kC, len - cs);
    __syncthreads();                                           // the previous chunk's tiles and weights are free
    if (warp == 0) gates(cnt);
    __syncthreads();
    commit();
    if (cs + kC < len) fetch(cs + kC);
    __syncthreads();
    // ---- outputs of the warp's 16 tokens
    const int r0 = warp * 16 + gq, r1 = r0 + 8;                 // rows of the chunk
    if (warp * 16 < cnt) {
      uint32_t qf[N / 16][4];
#pragma unroll
      for (int kk = 0; kk < N / 16; ++kk)
        ldmatrix_x4(qf[kk], smem_u32(sQ + (warp * 16 + (lane & 15)) * QP + (kk * 16 + (lane >> 4) * 8) * 2));
      float o[P / 8][4], den[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < P / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
      if (carried) {                                           // e^(m - M_i) Q [S | n], the memory as high + low halves
#pragma unroll
        for (int kk = 0; kk < N / 16; ++kk) {
          const float* s0 = sS + (kk * 16 + 2 * tq) * SP + gq;
#pragma unroll
          for (int nt = 0; nt < P / 8; ++nt) {
            uint32_t h0, l0, h1, l1;
            halves2<T>(s0[nt * 8], s0[SP + nt * 8], h0, l0);
            halves2<T>(s0[8 * SP + nt * 8], s0[9 * SP + nt * 8], h1, l1);
            mma_m16n8k16<T>(o[nt], qf[kk], h0, h1);
            mma_m16n8k16<T>(o[nt], qf[kk], l0, l1);
          }
          const float* n0 = sN + kk * 16 + 2 * tq;
          const T* e0 = reinterpret_cast<const T*>(&qf[kk][0]);     // row r0, columns 2 tq, 2 tq + 1
          const T* e1 = reinterpret_cast<const T*>(&qf[kk][1]);     // row r1
          const T* e2 = reinterpret_cast<const T*>(&qf[kk][2]);     // row r0, columns + 8
          const T* e3 = reinterpret_cast<const T*>(&qf[kk][3]);
          den[0] += to_f32(e0[0]) * n0[0] + to_f32(e0[1]) * n0[1] + to_f32(e2[0]) * n0[8] + to_f32(e2[1]) * n0[9];
          den[1] += to_f32(e1[0]) * n0[0] + to_f32(e1[1]) * n0[1] + to_f32(e3[0]) * n0[8] + to_f32(e3[1]) * n0[9];
        }
        const float w0 = sCar[r0], w1 = sCar[r1];
        den[0] *= w0; den[1] *= w1;
#pragma unroll
        for (int i = 0; i < P / 8; ++i) { o[i][0] *= w0; o[i][1] *= w0; o[i][2] *= w1; o[i][3] *= w1; }
      }
      // scores of the warp's rows against the keys up to its last row, weighted in fp32
      const float m0 = sM[r0], m1 = sM[r1];
      const int mj = lane >> 3, r = lane & 7;
      const uint32_t ka = smem_u32(sK) + ((mj >> 1) * 8 + r) * QP + (mj & 1) * 16;
      const uint32_t va = smem_u32(sV) + ((mj & 1) * 8 + r) * VP + (mj >> 1) * 16;
      for (int kt = 0; kt <= warp; ++kt) {
        float sc[2][4];
        sc[0][0] = sc[0][1] = sc[0][2] = sc[0][3] = sc[1][0] = sc[1][1] = sc[1][2] = sc[1][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < N / 16; ++kk) {
          uint32_t bfr[4];
          ldmatrix_x4(bfr, ka + kt * 16 * QP + kk * 32);
          mma_m16n8k16<T>(sc[0], qf[kk], bfr[0], bfr[1]);
          mma_m16n8k16<T>(sc[1], qf[kk], bfr[2], bfr[3]);
        }
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int key = kt * 16 + j * 8 + 2 * tq + (e & 1), row = (e >> 1) ? r1 : r0;
            const float w = key <= row ? fast_exp2(sA[key] - ((e >> 1) ? m1 : m0)) * a.q_scale : 0.f;   // keys past the end: a = -inf
            sc[j][e] *= w;
            den[e >> 1] += sc[j][e];
          }
        uint32_t ph[4], pl[4];
        halves2<T>(sc[0][0], sc[0][1], ph[0], pl[0]);
        halves2<T>(sc[0][2], sc[0][3], ph[1], pl[1]);
        halves2<T>(sc[1][0], sc[1][1], ph[2], pl[2]);
        halves2<T>(sc[1][2], sc[1][3], ph[3], pl[3]);
#pragma unroll
        for (int dn = 0; dn < P / 16; ++dn) {
          uint32_t bfr[4];
          ldmatrix_x4_trans(bfr, va + kt * 16 * VP + dn * 32);
          mma_m16n8k16<T>(o[2 * dn], ph, bfr[0], bfr[1]);
          mma_m16n8k16<T>(o[2 * dn + 1], ph, bfr[2], bfr[3]);
          mma_m16n8k16<T>(o[2 * dn], pl, bfr[0], bfr[1]);
          mma_m16n8k16<T>(o[2 * dn + 1], pl, bfr[2], bfr[3]);
        }
      }
#pragma unroll
      for (int r2 = 0; r2 < 2; ++r2) {                         // the four lanes of a row hold parts of its denominator
        den[r2] += __shfl_xor_sync(0xffffffffu, den[r2], 1);
        den[r2] += __shfl_xor_sync(0xffffffffu, den[r2], 2);
        den[r2] = 1.0f / (fmaxf(fabsf(den[r2]), sFloor[r2 ? r1 : r0]) + 1e-6f);
      }
      float* y0 = a.y + (int64_t)(start + cs + r0) * H * V + (int64_t)h * V + p0;
      float* y1 = a.y + (int64_t)(start + cs + r1) * H * V + (int64_t)h * V + p0;
      const bool pair = (V & 1) == 0;
#pragma unroll
      for (int i = 0; i < P / 8; ++i) {
        const int c = i * 8 + 2 * tq;
        const float a0 = o[i][0] * den[0], a1 = o[i][1] * den[0], b0 = o[i][2] * den[1], b1 = o[i][3] * den[1];
        if (pair) {
          if (r0 < cnt && c < pc) *reinterpret_cast<float2*>(y0 + c) = make_float2(a0, a1);
          if (r1 < cnt && c < pc) *reinterpret_cast<float2*>(y1 + c) = make_float2(b0, b1);
        } else {
          if (r0 < cnt && c < pc) y0[c] = a0;
          if (r0 < cnt && c + 1 < pc) y0[c + 1] = a1;
          if (r1 < cnt && c < pc) y1[c] = b0;
          if (r1 < cnt && c + 1 < pc) y1[c + 1] = b1;
        }
      }
    }
    __syncthreads();                                           // every warp is done with the old memory
    // ---- memory update: rows [16 mt, 16 mt + 16) of S and n per warp, 32 columns at a time
    const float dc = sScal[0];
    for (int mt = warp; mt < N / 16; mt += kChunkThreads / 32) {
      const int mj = lane >> 3, r = lane & 7;
      const uint32_t ka = smem_u32(sK) + ((mj >> 1) * 8 + r) * QP + (mt * 16 + (mj & 1) * 8) * 2;
      const uint32_t vh = smem_u32(sVh) + ((mj & 1) * 8 + r) * VP + (mj >> 1) * 16;
      const uint32_t vl = smem_u32(sVl) + ((mj & 1) * 8 + r) * VP + (mj >> 1) * 16;
      uint32_t af[kC / 16][4];
      float nn[2] = {0.f, 0.f};
#pragma unroll
      for (int kk = 0; kk < kC / 16; ++kk) {
        ldmatrix_x4_trans(af[kk], ka + kk * 16 * QP);
        // K^T fragment: rows gq / gq + 8 (memory rows), columns kk * 16 + 2 tq (+ 1, + 8, + 9) (tokens)
        const float* w0 = sW + kk * 16 + 2 * tq;
        const T* e0 = reinterpret_cast<const T*>(&af[kk][0]);
        const T* e1 = reinterpret_cast<const T*>(&af[kk][1]);
        const T* e2 = reinterpret_cast<const T*>(&af[kk][2]);
        const T* e3 = reinterpret_cast<const T*>(&af[kk][3]);
        nn[0] += to_f32(e0[0]) * w0[0] + to_f32(e0[1]) * w0[1] + to_f32(e2[0]) * w0[8] + to_f32(e2[1]) * w0[9];
        nn[1] += to_f32(e1[0]) * w0[0] + to_f32(e1[1]) * w0[1] + to_f32(e3[0]) * w0[8] + to_f32(e3[1]) * w0[9];
      }
#pragma unroll
      for (int r2 = 0; r2 < 2; ++r2) {
        nn[r2] += __shfl_xor_sync(0xffffffffu, nn[r2], 1);
        nn[r2] += __shfl_xor_sync(0xffffffffu, nn[r2], 2);
      }
      if (tq == 0) {
        float* np = sN + mt * 16 + gq;
        np[0] = dc * np[0] + nn[0];
        np[8] = dc * np[8] + nn[1];
      }
#pragma unroll
      for (int ng = 0; ng < P / 32; ++ng) {
        float acc[4][4];
        float* s0 = sS + (mt * 16 + gq) * SP + ng * 32 + 2 * tq;
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          acc[nt][0] = dc * s0[nt * 8]; acc[nt][1] = dc * s0[nt * 8 + 1];
          acc[nt][2] = dc * s0[8 * SP + nt * 8]; acc[nt][3] = dc * s0[8 * SP + nt * 8 + 1];
        }
#pragma unroll
        for (int kk = 0; kk < kC / 16; ++kk) {
          if (kk * 16 >= cnt) break;
#pragma unroll
          for (int pr = 0; pr < 2; ++pr) {
            uint32_t bh[4], bl[4];
            ldmatrix_x4_trans(bh, vh + kk * 16 * VP + (ng * 32 + pr * 16) * 2);
            ldmatrix_x4_trans(bl, vl + kk * 16 * VP + (ng * 32 + pr * 16) * 2);
            mma_m16n8k16<T>(acc[2 * pr], af[kk], bh[0], bh[1]);
            mma_m16n8k16<T>(acc[2 * pr + 1], af[kk], bh[2], bh[3]);
            mma_m16n8k16<T>(acc[2 * pr], af[kk], bl[0], bl[1]);
            mma_m16n8k16<T>(acc[2 * pr + 1], af[kk], bl[2], bl[3]);
          }
        }
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          s0[nt * 8] = acc[nt][0]; s0[nt * 8 + 1] = acc[nt][1];
          s0[8 * SP + nt * 8] = acc[nt][2]; s0[8 * SP + nt * 8 + 1] = acc[nt][3];
        }
      }
    }
    m = sScal[1];
    carried = true;
  }
  __syncthreads();
  for (int i = tid; i < D * P; i += kChunkThreads) {
    const int d = i / P, p = i - d * P;
    if (p < pc) st[(int64_t)d * V + p0 + p] = sS[d * SP + p];
  }
  if (last_tile(a.tickets + blockIdx.y * H + h, gridDim.z, &flag)) {
    for (int d = tid; d < D; d += kChunkThreads) st[(int64_t)D * V + d] = sN[d];
    if (tid == 0) st[(int64_t)D * V + D] = m;
  }
}

template <typename T>
int launch_scan(const MlstmArgs& a, int64_t num_seqs, cudaStream_t st) {
  const dim3 grid((unsigned)((a.V + kScanCols - 1) / kScanCols), (unsigned)a.H, (unsigned)num_seqs);
#define B2L_ML(R) b2l_launch(mlstm_scan_kernel<T, R>, grid, dim3(kScanThreads), (size_t)0, st, a)
  if (a.D <= 32) B2L_ML(2);
  else if (a.D <= 64) B2L_ML(4);
  else if (a.D <= 128) B2L_ML(8);
  else B2L_ML(16);
#undef B2L_ML
  B2L_LAUNCH_CHECK();
  return B2L_OK;
}

template <typename T, int N, int P>
int launch_chunk(const MlstmArgs& a, int64_t num_seqs, int vec, cudaStream_t st) {
  const size_t smem = (size_t)kC * (2 * (N + 8) + 3 * (P + 8)) * 2 + (size_t)(N * (P + 4) + N + 5 * kC + 4) * 4;
  static int cache[64] = {0};
  B2L_CUDA_CHECK(b2l_ensure_dynamic_smem(mlstm_chunk_kernel<T, N, P>, (int)smem, cache));
  b2l_launch(mlstm_chunk_kernel<T, N, P>, dim3((unsigned)a.H, (unsigned)num_seqs, (unsigned)((a.V + P - 1) / P)),
             dim3(kChunkThreads), smem, st, a, vec);
  B2L_LAUNCH_CHECK();
  return B2L_OK;
}

template <typename T>
int dispatch_chunk(const MlstmArgs& a, int64_t num_seqs, int vec, cudaStream_t st) {
  // 64 value columns per CTA, 32 when that leaves SMs without a CTA (the scores are then formed twice as often)
  const bool narrow = a.V <= 32 || (int64_t)a.H * num_seqs * ((a.V + 63) / 64) < b2l_num_sms();
#define B2L_MC(NN) return narrow ? launch_chunk<T, NN, 32>(a, num_seqs, vec, st) : launch_chunk<T, NN, 64>(a, num_seqs, vec, st)
  if (a.D <= 32) B2L_MC(32);
  if (a.D <= 64) B2L_MC(64);
  B2L_MC(128);
#undef B2L_MC
}

}  // namespace

/* Floats of one head's state block [S: dim x vdim | n: dim | m], padded to 16 bytes. */
extern "C" int64_t b2l_mlstm_head_floats(int dim, int vdim) { return ((int64_t)dim * vdim + dim + 1 + 3) / 4 * 4; }

/* chunked 0: token by token (any dtype, dim <= 256); 1: chunks of 64 tokens on the tensor cores (16-bit, dim <= 128).
 * tickets_i32: num_seqs * heads zeroed counters, left zeroed. */
extern "C" int b2l_mlstm(void* y_f32, void* state_f32, const void* q, int64_t q_row_stride, const void* k,
                         int64_t k_row_stride, const void* v, int64_t v_row_stride, const void* zi, int64_t zi_row_stride,
                         const void* zf, int64_t zf_row_stride, const void* bi, const void* bf, const void* seq_start,
                         const void* seq_ctx, const void* seq_slot, const void* seq_list, int64_t num_seqs, int heads,
                         int dim, int vdim, float q_scale, float gate_cap, void* tickets_i32, int64_t num_tickets,
                         int chunked, int dtype, void* stream) {
  B2L_REQUIRE(y_f32 && state_f32 && q && k && v && zi && zf && bi && bf && seq_start && seq_ctx && seq_slot && tickets_i32,
              "mlstm: null pointer");
  B2L_REQUIRE(heads > 0 && heads <= 65535 && dim > 0 && dim <= (chunked ? 128 : 256) && vdim > 0,
              "mlstm: %d heads, sizes %d x %d (chunked %d)", heads, dim, vdim, chunked);
  if (num_seqs <= 0) return B2L_OK;
  B2L_REQUIRE(num_seqs * heads <= num_tickets && num_seqs <= 65535, "mlstm: %lld sequences x %d heads need as many tickets (%lld)",
              (long long)num_seqs, heads, (long long)num_tickets);
  B2L_REQUIRE((uintptr_t)state_f32 % 16 == 0 && (uintptr_t)y_f32 % 8 == 0, "mlstm: state not aligned");
  MlstmArgs a;
  a.y = (float*)y_f32; a.state = (float*)state_f32; a.head_floats = b2l_mlstm_head_floats(dim, vdim);
  a.q = q; a.q_stride = q_row_stride; a.k = k; a.k_stride = k_row_stride; a.v = v; a.v_stride = v_row_stride;
  a.zi = zi; a.zi_stride = zi_row_stride; a.zf = zf; a.zf_stride = zf_row_stride; a.bi = bi; a.bf = bf;
  a.seq_start = (const int*)seq_start; a.seq_ctx = (const int*)seq_ctx; a.seq_slot = (const int*)seq_slot;
  a.seq_list = (const int*)seq_list; a.tickets = (int*)tickets_i32;
  a.H = heads; a.D = dim; a.V = vdim; a.q_scale = q_scale; a.cap = gate_cap;
  cudaStream_t st = (cudaStream_t)stream;
  if (chunked) {
    auto al = [](const void* p, int64_t stride) { return (uintptr_t)p % 16 == 0 && stride % 8 == 0; };
    const int vec = dim % 8 == 0 && vdim % 8 == 0 && al(q, q_row_stride) && al(k, k_row_stride) && al(v, v_row_stride);
    if (dtype == B2L_F16) return dispatch_chunk<__half>(a, num_seqs, vec, st);
    if (dtype == B2L_BF16) return dispatch_chunk<__nv_bfloat16>(a, num_seqs, vec, st);
    B2L_UNSUPPORTED("mlstm: chunks are for 16-bit activations (dtype %d)", dtype);
  }
  int rc = B2L_OK;
  B2L_DISPATCH_FLOAT(dtype, "mlstm", { rc = launch_scan<T>(a, num_seqs, st); });
  return rc;
}
