// Kernels of layers that carry SEVERAL residual streams x_1 .. x_S (fp32, [token, stream, channel])
// and connect each sublayer to all of them:
//
//   u   = sum_s in[s] x_s                       what a sublayer reads (through a norm)
//   x_t <- sum_s mix[s, t] x_s + out[t] * y     all streams at once, from the old ones
//
//   * hyper_update_(vec_)kernel  a sublayer's end in ONE pass over the streams: y put together from
//                            what the sublayer left (below), the new streams, the weighted sum the
//                            NEXT sublayer reads and its RMS norm.  Without y and mix it only reads:
//                            the first norm of a model, the norm behind the last layer (rows chosen).
//                            y = c0 w0[t] a0 + c1 w1[t] a1 + sum_k w[t, k] rows[pos[t, k]]: up to
//                            two dense terms with a constant and a factor a token, and the rows of a
//                            routed feed-forward's (token, choice) pairs, in the order chosen
//                            (a pair with position -1 has no row: an expert without matrices).
//                            All copies of a stream that is not split yet are ONE row: a stream
//                            stride of zero.
//   * bigram_embedding_kernel    x = E[token] * scale + P[row of (token before, token)]; the token
//                            before a portion's first one is per-request state.
// Arithmetic is fp32; T is the activation type (float for the 32-bit path, bf16 for serving).
#include "common.cuh"

namespace gf {

using bf = __nv_bfloat16;

struct HyperTerm {
  const void* a;            // [R, W] fp32 or bf16; null: no term
  int is_bf16;
  float c;
  const float* w;           // a factor a token (stride w_ld), or null
  int w_ld;
};

struct HyperArgs {
  const float* x;           // streams, or null
  long long x_tok, x_str;   // floats between tokens / streams
  int S, W;
  const float* mix;         // [S, S] from, to; null: no old streams in the new ones
  const float* out_w;       // [S]
  HyperTerm t0, t1;
  const float* pair_rows;   // [pairs, W] fp32, or null
  const int* pair_pos;      // [R, top]
  const float* pair_w;      // [R, top], or null: 1
  int top;
  int has_y;
  float* xo;                // new streams [R, S, W], or null
  const float* in_w;        // [S] what the next sublayer reads, or null: no norm
  const float* gamma;       // [W]
  float eps;
  void* normed;             // [R, W] of type T
  const int* rows;          // source rows (reading only), or null
};

__device__ __forceinline__ void term_quad(const HyperTerm& t, size_t r, int W, int j, float f,
                                          float (&y)[4]) {
  float v[4];
  if (t.is_bf16) Quad<bf>::load((const bf*)t.a + r * W + j, v);
  else Quad<float>::load((const float*)t.a + r * W + j, v);
#pragma unroll
  for (int i = 0; i < 4; ++i) y[i] = fmaf(f, v[i], y[i]);
}
__device__ __forceinline__ float term_factor(const HyperTerm& t, size_t r) {
  return t.a == nullptr ? 0.f : (t.w ? t.c * t.w[r * t.w_ld] : t.c);
}

// Up to SM streams, four channels an access, OPT quads a thread.  W % 4 == 0 and aligned rows.
template <typename T, int SM, int OPT>
__global__ void __launch_bounds__(1024)
hyper_update_vec_kernel(const HyperArgs a) {
  __shared__ float cm[SM * SM], co[SM], ci[SM], scratch[33];
  const int S = a.S, W = a.W, nq = W >> 2;
  pdl_trigger();
  if (threadIdx.x < SM * SM) {
    const int s = threadIdx.x / SM, t = threadIdx.x % SM;
    cm[threadIdx.x] = (a.mix && s < S && t < S) ? a.mix[s * S + t] : 0.f;
  }
  if (threadIdx.x < SM) {
    co[threadIdx.x] = (a.has_y && threadIdx.x < S) ? a.out_w[threadIdx.x] : 0.f;
    ci[threadIdx.x] = (a.in_w && threadIdx.x < S) ? a.in_w[threadIdx.x] : 0.f;
  }
  __syncthreads();
  pdl_wait();
  const size_t r = blockIdx.x, src = a.rows ? a.rows[r] : r;
  const float f0 = term_factor(a.t0, src), f1 = term_factor(a.t1, src);
  const float* xr = a.x ? a.x + src * a.x_tok : nullptr;
  const bool fresh = a.has_y || a.mix;             // new streams are formed (else only read)
  float u[OPT][4];
  float ss = 0.f;
#pragma unroll
  for (int o = 0; o < OPT; ++o) {
    const int q = threadIdx.x + o * blockDim.x;
#pragma unroll
    for (int i = 0; i < 4; ++i) u[o][i] = 0.f;
    if (q >= nq) continue;
    const int j = 4 * q;
    float xs[SM][4];
#pragma unroll
    for (int s = 0; s < SM; ++s) {
#pragma unroll
      for (int i = 0; i < 4; ++i) xs[s][i] = 0.f;
      if (s < S && xr) Quad<float>::load(xr + s * a.x_str + j, xs[s]);
    }
    if (!fresh) {
#pragma unroll
      for (int s = 0; s < SM; ++s)
#pragma unroll
        for (int i = 0; i < 4; ++i) u[o][i] = fmaf(ci[s], xs[s][i], u[o][i]);
    } else {
      float y[4] = {0.f, 0.f, 0.f, 0.f};
      if (a.pair_rows) {
        for (int k = 0; k < a.top; ++k) {
          const int p = fresh_index(a.pair_pos + src * a.top + k);
          if ((unsigned)p >= gridDim.x * (unsigned)a.top) continue;        // no row
          const float pw = a.pair_w ? a.pair_w[src * a.top + k] : 1.f;
          float v[4];
          Quad<float>::load(a.pair_rows + (size_t)p * W + j, v);
#pragma unroll
          for (int i = 0; i < 4; ++i) y[i] = fmaf(pw, v[i], y[i]);
        }
      }
      if (a.t0.a) term_quad(a.t0, src, W, j, f0, y);
      if (a.t1.a) term_quad(a.t1, src, W, j, f1, y);
#pragma unroll
      for (int t = 0; t < SM; ++t) {
        if (t >= S) continue;
        float n[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) n[i] = co[t] * y[i];
#pragma unroll
        for (int s = 0; s < SM; ++s)
#pragma unroll
          for (int i = 0; i < 4; ++i) n[i] = fmaf(cm[s * SM + t], xs[s][i], n[i]);
        if (a.xo) Quad<float>::store(a.xo + (r * S + t) * W + j, n);
#pragma unroll
        for (int i = 0; i < 4; ++i) u[o][i] = fmaf(ci[t], n[i], u[o][i]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) ss = fmaf(u[o][i], u[o][i], ss);
  }
  if (a.in_w == nullptr) return;
  ss = block_sum(ss, scratch);
  const float rms = sqrtf(ss / (float)W + a.eps);
  T* dst = (T*)a.normed + r * W;
#pragma unroll
  for (int o = 0; o < OPT; ++o) {
    const int q = threadIdx.x + o * blockDim.x;
    if (q >= nq) continue;
    float g[4];
    Quad<float>::load(a.gamma + 4 * q, g);
#pragma unroll
    for (int i = 0; i < 4; ++i) u[o][i] = u[o][i] / rms * g[i];
    Quad<T>::store(dst + 4 * q, u[o]);
  }
}

// Any number of streams and channels, a channel an access.  Shared memory: W floats.
template <typename T>
__global__ void hyper_update_kernel(const HyperArgs a) {
  extern __shared__ float row[];
  __shared__ float scratch[33];
  const int S = a.S, W = a.W;
  pdl_trigger();
  pdl_wait();
  const size_t r = blockIdx.x, src = a.rows ? a.rows[r] : r;
  const float f0 = term_factor(a.t0, src), f1 = term_factor(a.t1, src);
  const float* xr = a.x ? a.x + src * a.x_tok : nullptr;
  const bool fresh = a.has_y || a.mix;
  float ss = 0.f;
  for (int j = threadIdx.x; j < W; j += blockDim.x) {
    float y = 0.f, u = 0.f;
    if (a.pair_rows) {
      for (int k = 0; k < a.top; ++k) {
        const int p = fresh_index(a.pair_pos + src * a.top + k);
        if ((unsigned)p < gridDim.x * (unsigned)a.top)
          y = fmaf(a.pair_w ? a.pair_w[src * a.top + k] : 1.f, a.pair_rows[(size_t)p * W + j], y);
      }
    }
    auto term = [&](const HyperTerm& t, float f) {
      if (t.a)
        y = fmaf(f, t.is_bf16 ? to_f32(((const bf*)t.a)[src * W + j])
                              : ((const float*)t.a)[src * W + j], y);
    };
    term(a.t0, f0);
    term(a.t1, f1);
    for (int t = 0; t < S; ++t) {
      float n;
      if (!fresh) {
        n = xr[t * a.x_str + j];
      } else {
        n = a.has_y ? a.out_w[t] * y : 0.f;
        if (a.mix)
          for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], xr[s * a.x_str + j], n);
        if (a.xo) a.xo[(r * S + t) * W + j] = n;
      }
      if (a.in_w) u = fmaf(a.in_w[t], n, u);
    }
    row[j] = u;
    ss = fmaf(u, u, ss);
  }
  if (a.in_w == nullptr) return;
  ss = block_sum(ss, scratch);
  const float rms = sqrtf(ss / (float)W + a.eps);
  T* dst = (T*)a.normed + r * W;
  for (int j = threadIdx.x; j < W; j += blockDim.x) dst[j] = from_f32<T>(row[j] / rms * a.gamma[j]);
}

// A block a token.  state: the last token of earlier steps, one int a slot; the block that owns a
// portion's first token reads it and then writes the portion's last token (no other block touches
// the slot).  At position 0 there is no token before: row `buckets`.
template <typename W_>
__global__ void bigram_embedding_kernel(const int* __restrict__ ids, const W_* __restrict__ emb,
                                        float scale, const W_* __restrict__ table, int buckets,
                                        long long mul_prev, long long mul_cur,
                                        int* __restrict__ state, const int* __restrict__ positions,
                                        const int* __restrict__ seq_of_token,
                                        const int* __restrict__ cu_seqlens,
                                        const int* __restrict__ slot_ids, float* __restrict__ out,
                                        int H) {
  __shared__ int row_s;
  const int t = blockIdx.x;
  pdl_trigger();
  pdl_wait();
  const int cur = ids[t];
  if (threadIdx.x == 0) {
    const int b = seq_of_token[t];
    const bool first = t == cu_seqlens[b];
    int* slot = state + slot_ids[b];
    const int prev = first ? *slot : ids[t - 1];
    row_s = positions[t] == 0 ? buckets : (int)((prev * mul_prev + cur * mul_cur) % buckets);
    if (first) *slot = ids[cu_seqlens[b + 1] - 1];
  }
  __syncthreads();
  const W_* e = emb + (size_t)cur * H;
  const W_* p = table + (size_t)row_s * H;
  float* dst = out + (size_t)t * H;
  for (int j = threadIdx.x; j < H; j += blockDim.x)
    dst[j] = fmaf(to_f32(e[j]), scale, to_f32(p[j]));
}

}  // namespace gf

using namespace gf;

GF_DEFINE_PDL_SWITCH

// x null: no old streams (then mix is null); mix null with has_y == 0: only read.  t0 is fp32, t1 has
// t1_bf16.  Returns -4 for rows the kernels cannot hold, -2 for arguments that do not fit together.
GF_EXPORT int gf_hyper_update(const float* x, long long x_tok, long long x_str, int S, int W, int R,
                              const float* mix, const float* out_w, const float* t0, float c0,
                              const float* w0, int w0_ld, const void* t1, int t1_bf16, float c1,
                              const float* w1, int w1_ld, const float* pair_rows,
                              const int* pair_pos, const float* pair_w, int top, float* xo,
                              const float* in_w, const float* gamma, float eps, void* normed,
                              const int* rows, int dtype, void* stream) {
  if (R <= 0) return 0;
  HyperArgs a;
  a.x = x, a.x_tok = x_tok, a.x_str = x_str, a.S = S, a.W = W, a.mix = mix, a.out_w = out_w;
  a.t0 = HyperTerm{t0, 0, c0, w0, w0_ld};
  a.t1 = HyperTerm{t1, t1_bf16, c1, w1, w1_ld};
  a.pair_rows = pair_rows, a.pair_pos = pair_pos, a.pair_w = pair_w, a.top = top;
  a.has_y = t0 || t1 || pair_rows;
  a.xo = xo, a.in_w = in_w, a.gamma = gamma, a.eps = eps, a.normed = normed, a.rows = rows;
  if (S <= 0 || W <= 0 || (a.has_y && !out_w) || (mix && !x) || (!a.has_y && !mix && !x) ||
      (pair_rows && (!pair_pos || top <= 0)) || (in_w && (!gamma || !normed)) || (rows && xo))
    return -2;
  auto st = (cudaStream_t)stream;
  const bool quads = (((uintptr_t)x | (uintptr_t)t0 | (uintptr_t)t1 | (uintptr_t)pair_rows |
                       (uintptr_t)xo | (uintptr_t)gamma | (uintptr_t)normed) & 15) == 0 &&
                     W % 4 == 0 && x_tok % 4 == 0 && x_str % 4 == 0;
  const int nq = W / 4;
  if (quads && S <= 8 && nq <= 4096) {
    const int threads = nq >= 1024 ? 1024 : nq < 64 ? 64 : (nq + 31) / 32 * 32;
    const dim3 grid(R), block(threads);
#define GF_V(T, SM, OPT) return launch_kernel(hyper_update_vec_kernel<T, SM, OPT>, grid, block, 0, st, a)
#define GF_O(T, SM)                        \
  {                                        \
    if (nq <= threads) GF_V(T, SM, 1);     \
    if (nq <= 2 * threads) GF_V(T, SM, 2); \
    GF_V(T, SM, 4);                        \
  }
#define GF_S(T)             \
  {                         \
    if (S <= 2) GF_O(T, 2)  \
    if (S <= 4) GF_O(T, 4)  \
    GF_O(T, 8)              \
  }
    if (dtype == GF_F32) GF_S(float)
    GF_S(bf)
#undef GF_S
#undef GF_O
#undef GF_V
  }
  const size_t smem = (size_t)W * sizeof(float);
  if (smem > 48 * 1024) return -4;
  const dim3 grid(R), block(W >= 512 ? 256 : 128);
  if (dtype == GF_F32) return launch_kernel(hyper_update_kernel<float>, grid, block, smem, st, a);
  return launch_kernel(hyper_update_kernel<bf>, grid, block, smem, st, a);
}

GF_EXPORT int gf_bigram_embedding(const int* ids, const void* emb, float scale, const void* table,
                                  int buckets, long long mul_prev, long long mul_cur, int* state,
                                  const int* positions, const int* seq_of_token,
                                  const int* cu_seqlens, const int* slot_ids, float* out, int T,
                                  int H, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (buckets <= 0 || mul_prev < 0 || mul_cur < 0) return -2;
  auto st = (cudaStream_t)stream;
  const dim3 grid(T), block(H >= 1024 ? 256 : 128);
  if (dtype == GF_F32)
    return launch_kernel(bigram_embedding_kernel<float>, grid, block, 0, st, ids, (const float*)emb,
                         scale, (const float*)table, buckets, mul_prev, mul_cur, state, positions,
                         seq_of_token, cu_seqlens, slot_ids, out, H);
  return launch_kernel(bigram_embedding_kernel<bf>, grid, block, 0, st, ids, (const bf*)emb, scale,
                       (const bf*)table, buckets, mul_prev, mul_cur, state, positions, seq_of_token,
                       cu_seqlens, slot_ids, out, H);
}
