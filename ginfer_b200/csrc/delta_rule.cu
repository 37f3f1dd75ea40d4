// Gated delta rule with one decay per head and key channel, or one per head, over packed tokens of
// several requests.
// A request's state lives in a slot: S [heads, D, Vd] in fp32 and the last (taps - 1) inputs of the
// short convolutions, fp32 as well.
//
//   delta_prepare_kernel     a warp a (token, head): causal convolution over time (taps from the rows of
//                            this step, or from the slot where the step's portion starts later than
//                            the tap reaches) + SiLU on the q | k | v channels; q and k made unit
//                            vectors per head (q also times D^-1/2); decay g = exp(-exp(A_log_h) *
//                            softplus(a + dt_bias)); beta = sigmoid(b).  Everything leaves in fp32.
//   delta_prepare_heads_kernel  the same with one decay a head, four channels a lane, a warp walking
//                            over a run of tokens with the convolution's inputs in registers.
//   delta_conv_state_kernel  a thread a (request, channel): the slot's last inputs after the step.
//   delta_recurrence_kernel  per (request, head): S <- g * S (rows); u = beta (v - S^T k);
//                            S <- S + k u^T; o = S^T q, token after token.  The columns of S are
//                            independent: four lanes or a warp share a column (a share of the rows
//                            each, in registers).  The tokens' operands come through two stages of
//                            shared memory, a chunk ahead (cp.async).
//   delta_chunk_coef_kernel, delta_chunk_recurrence_kernel   the recurrence of long portions with one
//                            decay a head, eight tokens at a time (see there).
//   delta_output_kernel      a warp a (token, head): o / rms(o) * w * sigmoid(gate).
#include "common.cuh"

namespace gf {

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

struct DeltaDims {
  int H, G, D, Vd, taps;
  int channels;          // 2 G D + H Vd: the convolved columns q | k | v of a projection row
  int state_stride;      // floats a slot
  int conv_off;          // where the convolution inputs start in a slot
  int a_ld;              // one decay a head: floats between two tokens of its pre-activations
};

// ONE_DECAY: `a` holds a pre-activation a head (rows of a_ld floats), and one unit makes all heads'
// decays.  A warp a (token, unit): units 0 .. G-1 are q heads, G .. 2G-1 k heads, then H v heads, then H
// decay rows, then one unit for the betas.  No warp waits for another.
template <typename T>
__device__ __forceinline__ float conv_silu_at(const T* __restrict__ proj, int ld, int r, int i,
                                              const float* __restrict__ cs,
                                              const float* __restrict__ conv_w, int taps, int CH,
                                              int ch) {
  float acc = 0.f;
  for (int j = 0; j < taps; ++j) {
    const int off = i - (taps - 1 - j);           // place of the tap's input in the portion
    const float x = off >= 0 ? to_f32(proj[(size_t)(r - (taps - 1 - j)) * ld + ch])
                             : cs[(size_t)(taps - 1 + off) * CH + ch];
    acc = fmaf(conv_w[(size_t)ch * taps + j], x, acc);
  }
  return acc * sigmoid_f(acc);
}

constexpr int kPrepareWarps = 8;
constexpr int kPrepareMaxPerLane = 8;              // head sizes up to 256

template <typename T, bool ONE_DECAY>
__global__ void delta_prepare_kernel(const T* __restrict__ proj, int ld, int b_off,
                                     const float* __restrict__ a, const float* __restrict__ conv_w,
                                     const float* __restrict__ dt_bias,
                                     const float* __restrict__ A_log,
                                     const float* __restrict__ state,
                                     const int* __restrict__ seq_of_token,
                                     const int* __restrict__ cu_seqlens,
                                     const int* __restrict__ slot_ids, DeltaDims dm,
                                     float* __restrict__ qn, float* __restrict__ kn,
                                     float* __restrict__ v, float* __restrict__ g,
                                     float* __restrict__ beta) {
  const int r = blockIdx.x;
  const int unit = blockIdx.y * kPrepareWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_trigger();
  pdl_wait();
  const int G = dm.G, H = dm.H, D = dm.D, Vd = dm.Vd;
  if (unit >= 2 * G + H + (ONE_DECAY ? 0 : H) + 1) return;
  const int b = seq_of_token[r];
  const int i = r - cu_seqlens[b];                // place in this step's portion
  const float* cs = state + (size_t)slot_ids[b] * dm.state_stride + dm.conv_off;
  const int taps = dm.taps, CH = dm.channels, GD = G * D;
  if (unit < 2 * G) {                             // a q or k head: convolve, activate, unit vector
    const int ch0 = unit * D;                     // q heads and k heads follow one another
    float y[kPrepareMaxPerLane];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < kPrepareMaxPerLane; ++u) {
      const int d = lane + 32 * u;
      y[u] = d < D ? conv_silu_at(proj, ld, r, i, cs, conv_w, taps, CH, ch0 + d) : 0.f;
      ss += y[u] * y[u];
    }
    ss = warp_sum(ss);
    const bool is_q = unit < G;
    const float f = (is_q ? rsqrtf((float)D) : 1.f) / sqrtf(ss + 1e-6f);
    float* dst = (is_q ? qn : kn) + (size_t)r * GD + (size_t)(is_q ? unit : unit - G) * D;
#pragma unroll
    for (int u = 0; u < kPrepareMaxPerLane; ++u) {
      const int d = lane + 32 * u;
      if (d < D) dst[d] = y[u] * f;
    }
  } else if (unit < 2 * G + H) {                  // a v head
    const int h = unit - 2 * G;
    for (int j = lane; j < Vd; j += 32)
      v[((size_t)r * H + h) * Vd + j] =
          conv_silu_at(proj, ld, r, i, cs, conv_w, taps, CH, 2 * GD + h * Vd + j);
  } else if (!ONE_DECAY && unit < 2 * G + 2 * H) {              // a head's decays
    const int h = unit - 2 * G - H;
    const float rate = expf(A_log[h]);
    for (int d = lane; d < D; d += 32) {
      const size_t at = ((size_t)r * H + h) * D + d;
      g[at] = expf(-rate * softplus_f(a[at] + dt_bias[h * D + d]));
    }
  } else {
    for (int h = lane; h < H; h += 32)
      beta[(size_t)r * H + h] = sigmoid_f(to_f32(proj[(size_t)r * ld + b_off + h]));
    if (ONE_DECAY)
      for (int h = lane; h < H; h += 32)
        g[(size_t)r * H + h] =
            expf(-expf(A_log[h]) * softplus_f(a[(size_t)r * dm.a_ld + h] + dt_bias[h]));
  }
}

// One decay a head, the projection's row in fp32 (q | k | v first, decay and beta columns at a_off
// and b_off).  Units: G q heads, G k heads, H v heads, one for decays and betas.  A warp takes a unit
// and `run` consecutive tokens; lanes own four channels (NQ times); the last TAPS - 1 inputs stay in
// registers from token to token and come from the slot at a portion's start.  update_state (every
// portion of the step is one token): the same lanes bring the slot's inputs up to date.
// D, Vd, ld and the offsets are multiples of 4.
template <int TAPS, int NQ>
__global__ void __launch_bounds__(128)
delta_prepare_heads_kernel(const float* __restrict__ proj, int ld, int a_off, int b_off,
                           const float* __restrict__ conv_w, const float* __restrict__ dt_bias,
                           const float* __restrict__ A_log, float* __restrict__ state,
                           const int* __restrict__ seq_of_token,
                           const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids,
                           DeltaDims dm, int T, int run, int update_state, float* __restrict__ qn,
                           float* __restrict__ kn, float* __restrict__ v, float* __restrict__ g,
                           float* __restrict__ beta) {
  constexpr int KEEP = TAPS - 1;
  const int lane = threadIdx.x & 31;
  const int G = dm.G, H = dm.H, D = dm.D, Vd = dm.Vd, GD = G * D;
  const int unit = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int r0 = blockIdx.x * run, r1 = min(r0 + run, T);
  const bool convolves = unit < 2 * G + H;
  const int size = unit < 2 * G ? D : Vd;
  const int ch0 = unit < 2 * G ? unit * D : 2 * GD + (unit - 2 * G) * Vd;
  float w[NQ][4][TAPS];
  if (convolves) {                                  // weights: before the wait
#pragma unroll
    for (int u = 0; u < NQ; ++u)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int d = 4 * (lane + 32 * u) + i;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[u][i][j] = d < size ? conv_w[(size_t)(ch0 + d) * TAPS + j] : 0.f;
      }
  }
  // few tokens: the recurrence may start early.  In a prompt its long-lived blocks would land several
  // to an SM on the first SMs that drain.
  if (run == 1) pdl_trigger();
  pdl_wait();
  if (unit > 2 * G + H) return;
  if (!convolves) {
    for (int e = lane; e < (r1 - r0) * H; e += 32) {
      const int r = r0 + e / H, h = e % H;
      const float* row = proj + (size_t)r * ld;
      beta[(size_t)r * H + h] = sigmoid_f(row[b_off + h]);
      g[(size_t)r * H + h] = expf(-expf(A_log[h]) * softplus_f(row[a_off + h] + dt_bias[h]));
    }
    return;
  }
  float past[NQ][4][KEEP > 0 ? KEEP : 1];           // inputs of the tokens before, oldest first
  for (int r = r0; r < r1; ++r) {
    const int b = seq_of_token[r], start = cu_seqlens[b];
    float* cs = state + (size_t)slot_ids[b] * dm.state_stride + dm.conv_off;
    if (r == r0 || r == start) {
#pragma unroll
      for (int m = 0; m < KEEP; ++m) {
        const int at = r - KEEP + m;                // the row of this input, if the step has it
#pragma unroll
        for (int u = 0; u < NQ; ++u) {
          const int d = 4 * (lane + 32 * u);
          float x[4] = {0.f, 0.f, 0.f, 0.f};
          if (d < size)
            Quad<float>::load(at >= start ? proj + (size_t)at * ld + ch0 + d
                                          : cs + (size_t)(KEEP + at - start) * dm.channels + ch0 + d,
                              x);
#pragma unroll
          for (int i = 0; i < 4; ++i) past[u][i][m] = x[i];
        }
      }
    }
    float y[NQ][4];
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < NQ; ++u) {
      const int d = 4 * (lane + 32 * u);
      float x[4] = {0.f, 0.f, 0.f, 0.f};
      if (d < size) Quad<float>::load(proj + (size_t)r * ld + ch0 + d, x);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        float acc = 0.f;
#pragma unroll
        for (int m = 0; m < KEEP; ++m) acc = fmaf(w[u][i][m], past[u][i][m], acc);
        acc = fmaf(w[u][i][KEEP], x[i], acc);
        y[u][i] = acc * sigmoid_f(acc);
        ss += y[u][i] * y[u][i];
#pragma unroll
        for (int m = 0; m + 1 < KEEP; ++m) past[u][i][m] = past[u][i][m + 1];
        if (KEEP > 0) past[u][i][KEEP > 0 ? KEEP - 1 : 0] = x[i];
      }
      if (update_state && d < size) {
#pragma unroll
        for (int m = 0; m < KEEP; ++m) {
          const float s4[4] = {past[u][0][m], past[u][1][m], past[u][2][m], past[u][3][m]};
          Quad<float>::store(cs + (size_t)m * dm.channels + ch0 + d, s4);
        }
      }
    }
    float f = 1.f;
    float* dst;
    if (unit < 2 * G) {
      const bool is_q = unit < G;
      ss = warp_sum(ss);
      f = (is_q ? rsqrtf((float)D) : 1.f) / sqrtf(ss + 1e-6f);
      dst = (is_q ? qn : kn) + (size_t)r * GD + (size_t)(is_q ? unit : unit - G) * D;
    } else {
      dst = v + ((size_t)r * H + (unit - 2 * G)) * Vd;
    }
#pragma unroll
    for (int u = 0; u < NQ; ++u) {
      const int d = 4 * (lane + 32 * u);
      if (d < size) {
        const float o4[4] = {y[u][0] * f, y[u][1] * f, y[u][2] * f, y[u][3] * f};
        Quad<float>::store(dst + d, o4);
      }
    }
  }
}

template <typename T>
__global__ void delta_conv_state_kernel(const T* __restrict__ proj, int ld,
                                        float* __restrict__ state,
                                        const int* __restrict__ cu_seqlens,
                                        const int* __restrict__ slot_ids, DeltaDims dm) {
  const int b = blockIdx.y;
  const int ch = blockIdx.x * blockDim.x + threadIdx.x;
  pdl_trigger();
  pdl_wait();
  if (ch >= dm.channels) return;
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  float* cs = state + (size_t)slot_ids[b] * dm.state_stride + dm.conv_off;
  const int keep = dm.taps - 1;
  // entry m holds the input (keep - m) tokens before the next one; ascending m reads entries that
  // are not yet overwritten
  for (int m = 0; m < keep; ++m) {
    const int i = n - keep + m;
    cs[(size_t)m * dm.channels + ch] =
        i >= 0 ? to_f32(proj[(size_t)(start + i) * ld + ch]) : cs[(size_t)(m + n) * dm.channels + ch];
  }
}

constexpr int kRecurrenceThreads = 128;
constexpr int kMaxColumnsPerBlock = 32;
constexpr int kStages = 3;             // chunks of tokens in shared memory

__device__ __forceinline__ void copy_async_4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void copy_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// A block = (request, head, 128 / LP columns of S); LP lanes share a column, DPER rows each.  The
// tokens' k, q, g rows (padded to Dp = LP * DPER floats, the padding zero), the block's v columns and
// beta come through three stages of shared memory, CHUNK tokens each, asked for two chunks ahead
// with cp.async.  LP = 4 where requests x heads x columns fill the device (decode batches); LP = 32
// (a warp a column, eight columns a block) where they do not (one long prompt): a token is a chain
// of dependent instructions for a warp, and with eight times the lanes a column the chain is short
// and eight times as many warps share an SM's schedulers.
// ONE_DECAY: g holds a decay a head; it travels beside beta.
template <int DPER, int LP, int CHUNK, int THREADS, bool ONE_DECAY>
__global__ void __launch_bounds__(THREADS)
delta_recurrence_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                        const float* __restrict__ v, const float* __restrict__ g,
                        const float* __restrict__ beta, float* __restrict__ state,
                        const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids,
                        DeltaDims dm, float* __restrict__ o) {
  constexpr int Dp = LP * DPER;
  constexpr int kV = (ONE_DECAY ? 2 : 3) * Dp;                 // where a token's v columns start
  constexpr int kB = kV + kMaxColumnsPerBlock;                 // beta (and the head's decay)
  constexpr int kTok = kB + 4;                                 // floats a token in a stage
  extern __shared__ __align__(16) float stage[];               // [kStages][CHUNK][kTok]
  constexpr int cols = THREADS / LP;
  const int b = blockIdx.x / dm.H, h = blockIdx.x - b * dm.H;
  const int part = threadIdx.x % LP, lc = threadIdx.x / LP;
  const int col0 = blockIdx.y * cols, col = col0 + lc;
  pdl_trigger();
  const int D = dm.D, Vd = dm.Vd;
  for (int i = threadIdx.x; i < kStages * CHUNK * kTok; i += blockDim.x) stage[i] = 0.f;
  __syncthreads();
  pdl_wait();
  const int row0 = part * DPER;
  const bool col_ok = col < Vd;
  const int cj = col_ok ? col : 0;
  const int kvh = h / (dm.H / dm.G);
  float* Sg = state + (size_t)slot_ids[b] * dm.state_stride + ((size_t)h * D) * Vd + cj;
  float S[DPER];
#pragma unroll
  for (int i = 0; i < DPER; ++i) S[i] = (row0 + i < D) ? Sg[(size_t)(row0 + i) * Vd] : 0.f;
  const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
  const size_t GD = (size_t)dm.G * D, HD = (size_t)dm.H * D, HV = (size_t)dm.H * Vd;
  const int ncols = min(cols, Vd - col0);
  // 16-byte copies where rows allow it (a thread keeps the same piece of every token), else 4-byte
  const bool vec = (D & 3) == 0 && (Vd & 3) == 0 && (ncols & 3) == 0;
  const int dq = D >> 2, nd = (ONE_DECAY ? 2 : 3) * dq, pieces = nd + (ncols >> 2);
  auto ask = [&](int chunk) {                      // the chunk's tokens into stage chunk % kStages
    float* st = stage + (size_t)(chunk % kStages) * CHUNK * kTok;
    const int ta = t0 + chunk * CHUNK, n = min(CHUNK, t1 - ta);
    if (vec) {
      for (int e = threadIdx.x; e < pieces; e += blockDim.x) {
        const float* src;
        int dst, step;                             // source floats from one token to the next
        if (e < dq) src = kn + (size_t)ta * GD + (size_t)kvh * D + 4 * e, dst = 4 * e, step = (int)GD;
        else if (e < 2 * dq)
          src = qn + (size_t)ta * GD + (size_t)kvh * D + 4 * (e - dq), dst = Dp + 4 * (e - dq), step = (int)GD;
        else if (!ONE_DECAY && e < nd)
          src = g + (size_t)ta * HD + (size_t)h * D + 4 * (e - 2 * dq), dst = 2 * Dp + 4 * (e - 2 * dq),
          step = (int)HD;
        else
          src = v + (size_t)ta * HV + (size_t)h * Vd + col0 + 4 * (e - nd),
          dst = kV + 4 * (e - nd), step = (int)HV;
        for (int tt = 0; tt < n; ++tt)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(
                           smem_u32(st + (size_t)tt * kTok + dst)),
                       "l"(src + (size_t)tt * step)
                       : "memory");
      }
      if (threadIdx.x < n) {
        copy_async_4(st + (size_t)threadIdx.x * kTok + kB,
                     beta + (size_t)(ta + threadIdx.x) * dm.H + h);
        if (ONE_DECAY)
          copy_async_4(st + (size_t)threadIdx.x * kTok + kB + 1,
                       g + (size_t)(ta + threadIdx.x) * dm.H + h);
      }
    } else {
      const int rd = (ONE_DECAY ? 2 : 3) * D;
      const int per = rd + ncols + (ONE_DECAY ? 2 : 1);
      for (int i = threadIdx.x; i < n * per; i += blockDim.x) {
        const int tt = i / per, e = i - tt * per;
        const size_t t = (size_t)(ta + tt);
        float* dst = st + (size_t)tt * kTok;
        if (e < D) copy_async_4(dst + e, kn + t * GD + (size_t)kvh * D + e);
        else if (e < 2 * D) copy_async_4(dst + Dp + (e - D), qn + t * GD + (size_t)kvh * D + (e - D));
        else if (!ONE_DECAY && e < rd) copy_async_4(dst + 2 * Dp + (e - 2 * D), g + t * HD + (size_t)h * D + (e - 2 * D));
        else if (e < rd + ncols)
          copy_async_4(dst + kV + (e - rd), v + t * HV + (size_t)h * Vd + col0 + (e - rd));
        else if (e == rd + ncols) copy_async_4(dst + kB, beta + t * dm.H + h);
        else copy_async_4(dst + kB + 1, g + t * dm.H + h);
      }
    }
    copy_async_commit();
  };
  const int nchunks = (t1 - t0 + CHUNK - 1) / CHUNK;
  // two chunks are under way while a third is worked on (a group is committed every turn, empty
  // ones too, so that "all but the last two" always means "chunk c has landed")
  for (int c = 0; c < kStages - 1; ++c) {
    if (c < nchunks) ask(c);
    else copy_async_commit();
  }
  for (int c = 0; c < nchunks; ++c) {
    // the stage of chunk c + 2 held chunk c - 1, which every warp left at the last barrier
    if (c + kStages - 1 < nchunks) ask(c + kStages - 1);
    else copy_async_commit();
    copy_async_wait<kStages - 1>();
    __syncthreads();
    const float* st = stage + (size_t)(c % kStages) * CHUNK * kTok;
    const int ta = t0 + c * CHUNK, n = min(CHUNK, t1 - ta);
    // The chunk's tokens, unrolled: the read-out o = S^T q of a token is off the chain that the
    // next token waits for (only u is on it), so its lane reduction is left until the chunk is
    // done and the eight reductions run side by side.
    float outp[CHUNK];
#pragma unroll
    for (int tt = 0; tt < CHUNK; ++tt) {
      outp[tt] = 0.f;
      if (tt < n) {
        const float* tok = st + (size_t)tt * kTok;
        const float4* k4 = reinterpret_cast<const float4*>(tok + row0);
        const float4* q4 = reinterpret_cast<const float4*>(tok + Dp + row0);
        const float4* g4 = reinterpret_cast<const float4*>(tok + 2 * Dp + row0);   // (not ONE_DECAY)
        const float vc = tok[kV + lc], bc = tok[kB], g1 = tok[kB + 1];
        float kc[DPER];
#pragma unroll
        for (int i = 0; i < DPER / 4; ++i) {
          const float4 kk = k4[i];
          const float4 gg = ONE_DECAY ? make_float4(g1, g1, g1, g1) : g4[i];
          kc[4 * i] = kk.x, kc[4 * i + 1] = kk.y, kc[4 * i + 2] = kk.z, kc[4 * i + 3] = kk.w;
          S[4 * i] *= gg.x, S[4 * i + 1] *= gg.y, S[4 * i + 2] *= gg.z, S[4 * i + 3] *= gg.w;
        }
        float d4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < DPER; ++i) d4[i & 3] = fmaf(S[i], kc[i], d4[i & 3]);
        float dot = (d4[0] + d4[1]) + (d4[2] + d4[3]);
#pragma unroll
        for (int sh = 1; sh < LP; sh <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, sh);
        const float u = bc * (vc - dot);
        float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < DPER / 4; ++i) {
          const float4 qq = q4[i];
          S[4 * i] = fmaf(kc[4 * i], u, S[4 * i]);
          S[4 * i + 1] = fmaf(kc[4 * i + 1], u, S[4 * i + 1]);
          S[4 * i + 2] = fmaf(kc[4 * i + 2], u, S[4 * i + 2]);
          S[4 * i + 3] = fmaf(kc[4 * i + 3], u, S[4 * i + 3]);
          o4[0] = fmaf(S[4 * i], qq.x, o4[0]);
          o4[1] = fmaf(S[4 * i + 1], qq.y, o4[1]);
          o4[2] = fmaf(S[4 * i + 2], qq.z, o4[2]);
          o4[3] = fmaf(S[4 * i + 3], qq.w, o4[3]);
        }
        outp[tt] = (o4[0] + o4[1]) + (o4[2] + o4[3]);
      }
    }
#pragma unroll
    for (int sh = 1; sh < LP; sh <<= 1) {
#pragma unroll
      for (int tt = 0; tt < CHUNK; ++tt) outp[tt] += __shfl_xor_sync(0xffffffffu, outp[tt], sh);
    }
    if (part == 0 && col_ok) {
#pragma unroll
      for (int tt = 0; tt < CHUNK; ++tt)
        if (tt < n) o[(size_t)(ta + tt) * HV + (size_t)h * Vd + col] = outp[tt];
    }
    __syncthreads();                               // the stage is free for the chunk after next
  }
  if (col_ok) {
#pragma unroll
    for (int i = 0; i < DPER; ++i)
      if (row0 + i < D) Sg[(size_t)(row0 + i) * Vd] = S[i];
  }
}

// ---- eight tokens at a time ---------------------------------------------------------------------
// With one decay a head the recurrence over a chunk of tokens 0 .. 7 that starts from S needs S only
// in products that do not wait for one another.  With G_i = g_0 .. g_i, R(j, i) = g_(j+1) .. g_i:
//
//   u_i = beta_i (v_i - G_i S^T k_i) - sum_(j<i) L_ij u_j,   L_ij = beta_i R(j, i) k_j.k_i
//   o_i = G_i S^T q_i + sum_(j<=i) M_ij u_j,                 M_ij = R(j, i) k_j.q_i
//   S  <- G_7 S + sum_j R(j, 7) k_j u_j^T
//
// (ratios of decays are products of the factors between the two tokens, never quotients).  The chain
// from token to token is then eight multiply-adds in registers a chunk, instead of a pass over S and a
// reduction across lanes a token.  Everything is 32-bit multiply-adds.
constexpr int CT = 8;                                          // tokens a chunk
constexpr int kCoefL = 0, kCoefM = 64, kCoefG = 128, kCoefE = 136, kCoefBeta = 144, kCoefs = 152;

// Chunks of request b start at the packed number cu[b] / CT + b; no two requests' chunks meet.
__device__ __forceinline__ int chunk_number(int first_row, int b, int c) { return first_row / CT + b + c; }

// A warp a (chunk, kv head): the 64 dot products k_j.k_i (j < i) and k_j.q_i (j <= i), then for every
// head of the group L, M, G, E (E_j = R(j, 7)) and beta.  Tokens behind the portion's end count as
// k = q = 0, g = 1, beta = 0.
__global__ void __launch_bounds__(128)
delta_chunk_coef_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                        const float* __restrict__ g, const float* __restrict__ beta,
                        const int* __restrict__ cu_seqlens, DeltaDims dm, float* __restrict__ coef) {
  const int lane = threadIdx.x & 31;
  const int c = blockIdx.x * 4 + (threadIdx.x >> 5), b = blockIdx.y, kvh = blockIdx.z;
  pdl_wait();
  const int t0 = cu_seqlens[b], ta = t0 + c * CT, n = min(CT, cu_seqlens[b + 1] - ta);
  if (n <= 0) return;
  const int D = dm.D, H = dm.H, per = H / dm.G;
  const size_t GD = (size_t)dm.G * D;
  // pair (a, e) = (m / 8, m % 8): k_e.k_a for a > e, k_a.q_e for a <= e
  float val[64];
#pragma unroll
  for (int m = 0; m < 64; ++m) val[m] = 0.f;
  for (int d = 4 * lane; d < D; d += 128) {
    float k[CT][4], q[CT][4];
#pragma unroll
    for (int i = 0; i < CT; ++i) {
#pragma unroll
      for (int x = 0; x < 4; ++x) k[i][x] = q[i][x] = 0.f;
      if (i < n) {
        const size_t at = (size_t)(ta + i) * GD + (size_t)kvh * D + d;
        Quad<float>::load(kn + at, k[i]);
        Quad<float>::load(qn + at, q[i]);
      }
    }
#pragma unroll
    for (int m = 0; m < 64; ++m) {
      const int a = m >> 3, e = m & 7;
#pragma unroll
      for (int x = 0; x < 4; ++x) val[m] = fmaf(k[a > e ? e : a][x], a > e ? k[a][x] : q[e][x], val[m]);
    }
  }
  // add up across the lanes, halving the values each lane carries: lane l ends with m = l, l + 32
#pragma unroll
  for (int half = 16; half >= 1; half >>= 1) {
    const bool up = lane & half;
    // values that differ in this bit of m are neighbours at distance `half`; what is left of the
    // list is indexed by m with the higher bits already fixed to the lane's
#pragma unroll
    for (int hi = 0; hi < 2; ++hi)
#pragma unroll
      for (int m = 0; m < half; ++m) {
        const float lo_v = val[32 * hi + m], hi_v = val[32 * hi + m + half];
        const float got = __shfl_xor_sync(0xffffffffu, up ? lo_v : hi_v, half);
        val[32 * hi + m] = (up ? hi_v : lo_v) + got;
      }
  }
  const float mine[2] = {val[0], val[32]};
  float* base = coef + ((size_t)chunk_number(t0, b, c) * H + (size_t)kvh * per) * kCoefs;
  for (int hh = 0; hh < per; ++hh) {
    const int h = kvh * per + hh;
    const bool real = lane < n;
    const float gl = real ? g[(size_t)(ta + lane) * H + h] : 1.f;
    const float bl = real ? beta[(size_t)(ta + lane) * H + h] : 0.f;
    float* dst = base + (size_t)hh * kCoefs;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int m = lane + 32 * x, a = m >> 3, e = m & 7;
      const int i = a > e ? a : e, j = a > e ? e : a;          // j <= i
      float r = 1.f;
#pragma unroll
      for (int s = 1; s < CT; ++s) {
        const float gs = __shfl_sync(0xffffffffu, gl, s);
        if (s > j && s <= i) r *= gs;
      }
      const float bi = __shfl_sync(0xffffffffu, bl, i);
      if (a > e) {
        dst[kCoefL + i * CT + j] = bi * r * mine[x];
        dst[kCoefM + j * CT + i] = 0.f;                         // (M is read as whole rows)
      } else {
        dst[kCoefM + i * CT + j] = r * mine[x];
        if (i == j) dst[kCoefL + i * CT + j] = 0.f;
      }
    }
    float G = 1.f, E = 1.f;
#pragma unroll
    for (int s = 0; s < CT; ++s) {
      const float gs = __shfl_sync(0xffffffffu, gl, s);
      if (s <= lane) G *= gs;
      if (s > lane) E *= gs;
    }
    if (lane < CT) {
      dst[kCoefG + lane] = G;
      dst[kCoefE + lane] = E;
      dst[kCoefBeta + lane] = bl;
    }
  }
}

// A block = (request, head, 16 columns of S); LANES (8 or 16) lanes a column.  Lane p of a column owns
// the rows 4 (p + LANES i) .. + 3, i < DPER / 4, so that the lanes' reads of a token's k and q are one run of
// shared memory.  Stages as in the kernel above, one barrier a chunk.
template <int DPER, int LANES>
__global__ void __launch_bounds__(16 * LANES)
delta_chunk_recurrence_kernel(const float* __restrict__ qn, const float* __restrict__ kn,
                              const float* __restrict__ v, const float* __restrict__ coef,
                              float* __restrict__ state, const int* __restrict__ cu_seqlens,
                              const int* __restrict__ slot_ids, DeltaDims dm, float* __restrict__ o) {
  constexpr int Dp = LANES * DPER, COLS = 16, NQ = DPER / 4;
  constexpr int kQ = CT * Dp, kVc = 2 * CT * Dp, kC = kVc + CT * COLS, kStage = kC + kCoefs;
  extern __shared__ __align__(16) float stage[];               // [kStages][kStage]
  const int b = blockIdx.x / dm.H, h = blockIdx.x - b * dm.H;
  const int p = threadIdx.x % LANES, lc = threadIdx.x / LANES;
  const int col0 = blockIdx.y * COLS, col = col0 + lc;
  pdl_trigger();
  const int D = dm.D, Vd = dm.Vd;
  for (int i = threadIdx.x; i < kStages * kStage; i += blockDim.x) stage[i] = 0.f;
  __syncthreads();
  pdl_wait();
  const bool col_ok = col < Vd;
  const int cj = col_ok ? col : 0;
  const int kvh = h / (dm.H / dm.G);
  float* Sg = state + (size_t)slot_ids[b] * dm.state_stride + ((size_t)h * D) * Vd + cj;
  float S[NQ][4];
#pragma unroll
  for (int i = 0; i < NQ; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = 4 * (p + LANES * i) + x;
      S[i][x] = row < D ? Sg[(size_t)row * Vd] : 0.f;
    }
  const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
  const size_t GD = (size_t)dm.G * D, HV = (size_t)dm.H * Vd;
  const int vq = min(COLS, Vd - col0) >> 2, dq = D >> 2;
  const int nchunks = (t1 - t0 + CT - 1) / CT;
  const float* coef0 = coef + ((size_t)chunk_number(t0, b, 0) * dm.H + h) * kCoefs;
  auto copy16 = [](float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  };
  auto ask = [&](int c) {
    float* st = stage + (size_t)(c % kStages) * kStage;
    const int ta = t0 + c * CT, n = min(CT, t1 - ta);
    for (int e = threadIdx.x; e < n * dq; e += blockDim.x) {
      const int t = e / dq, d = 4 * (e - t * dq);
      const size_t at = (size_t)(ta + t) * GD + (size_t)kvh * D + d;
      copy16(st + t * Dp + d, kn + at);
      copy16(st + kQ + t * Dp + d, qn + at);
    }
    for (int e = threadIdx.x; e < n * vq; e += blockDim.x) {
      const int t = e / vq, d = 4 * (e - t * vq);
      copy16(st + kVc + t * COLS + d, v + (size_t)(ta + t) * HV + (size_t)h * Vd + col0 + d);
    }
    for (int e = threadIdx.x; e < kCoefs / 4; e += blockDim.x)
      copy16(st + kC + 4 * e, coef0 + (size_t)c * dm.H * kCoefs + 4 * e);
  };
  for (int c = 0; c < kStages - 1; ++c) {
    if (c < nchunks) ask(c);
    copy_async_commit();
  }
  for (int c = 0; c < nchunks; ++c) {
    copy_async_wait<kStages - 2>();
    __syncthreads();                 // chunk c has landed for all, and all have left chunk c - 1
    if (c + kStages - 1 < nchunks) ask(c + kStages - 1);       // into the stage of chunk c - 1
    copy_async_commit();
    const float* st = stage + (size_t)(c % kStages) * kStage;
    const float* cf = st + kC;
    // this lane's share of S^T k_i (x[i]) and S^T q_i (x[8 + i])
    float x[2 * CT];
#pragma unroll
    for (int i = 0; i < 2 * CT; ++i) x[i] = 0.f;
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const float* at = st + 4 * (p + LANES * i);
#pragma unroll
      for (int t = 0; t < 2 * CT; ++t) {
        const float4 a = *reinterpret_cast<const float4*>(at + t * Dp);
        x[t] = fmaf(S[i][0], a.x, fmaf(S[i][1], a.y, fmaf(S[i][2], a.z, fmaf(S[i][3], a.w, x[t]))));
      }
    }
    // add up across the column's lanes: of eight, lane p ends with both sums of token p; of sixteen,
    // lane p with S^T k of token p or S^T q of token p - 8
#pragma unroll
    for (int half = LANES / 2; half >= 1; half >>= 1) {
      const bool up = p & half;
#pragma unroll
      for (int hi = 0; hi < 2 * CT / LANES; ++hi)
#pragma unroll
        for (int m = 0; m < half; ++m) {
          const float lo_v = x[LANES * hi + m], hi_v = x[LANES * hi + m + half];
          const float got = __shfl_xor_sync(0xffffffffu, up ? lo_v : hi_v, half);
          x[LANES * hi + m] = (up ? hi_v : lo_v) + got;
        }
    }
    const int tok = p % CT;                                     // the token this lane looks after
    const float Gp = cf[kCoefG + tok];
    const float rp = cf[kCoefBeta + tok] * (st[kVc + tok * COLS + lc] - Gp * x[0]);
    float u[CT];
#pragma unroll
    for (int i = 0; i < CT; ++i) u[i] = __shfl_sync(0xffffffffu, rp, i, LANES);
#pragma unroll
    for (int j = 0; j < CT - 1; ++j)
#pragma unroll
      for (int i = j + 1; i < CT; ++i) u[i] = fmaf(-cf[kCoefL + i * CT + j], u[j], u[i]);
    {
      const float4* Mp = reinterpret_cast<const float4*>(cf + kCoefM + tok * CT);
      const float4 m0 = Mp[0], m1 = Mp[1];
      float out = Gp * (LANES == CT ? x[CT] : x[0]);
      out = fmaf(m0.x, u[0], fmaf(m0.y, u[1], fmaf(m0.z, u[2], fmaf(m0.w, u[3], out))));
      out = fmaf(m1.x, u[4], fmaf(m1.y, u[5], fmaf(m1.z, u[6], fmaf(m1.w, u[7], out))));
      const int row = t0 + c * CT + tok;
      if (col_ok && row < t1 && p >= LANES - CT) o[(size_t)row * HV + (size_t)h * Vd + col] = out;
    }
    const float Gc = cf[kCoefG + CT - 1];
#pragma unroll
    for (int j = 0; j < CT; ++j) u[j] *= cf[kCoefE + j];
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const float* at = st + 4 * (p + LANES * i);
#pragma unroll
      for (int y = 0; y < 4; ++y) S[i][y] *= Gc;
#pragma unroll
      for (int t = 0; t < CT; ++t) {
        const float4 a = *reinterpret_cast<const float4*>(at + t * Dp);
        S[i][0] = fmaf(a.x, u[t], S[i][0]);
        S[i][1] = fmaf(a.y, u[t], S[i][1]);
        S[i][2] = fmaf(a.z, u[t], S[i][2]);
        S[i][3] = fmaf(a.w, u[t], S[i][3]);
      }
    }
  }
  if (col_ok) {
#pragma unroll
    for (int i = 0; i < NQ; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int row = 4 * (p + LANES * i) + x;
        if (row < D) Sg[(size_t)row * Vd] = S[i][x];
      }
  }
}

template <int DPER, int LANES>
static int launch_chunks(const float* qn, const float* kn, const float* v, const float* coef,
                         float* state, const int* cu_seqlens, const int* slot_ids, int B,
                         const DeltaDims& dm, float* o, cudaStream_t st) {
  const size_t smem = (size_t)kStages * (2 * CT * LANES * DPER + CT * 16 + kCoefs) * sizeof(float);
  static OncePerDevice attrs;
  if (int rc = attrs.run([&] {
        return cudaFuncSetAttribute(delta_chunk_recurrence_kernel<DPER, LANES>,
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      }))
    return rc;
  return launch_kernel(delta_chunk_recurrence_kernel<DPER, LANES>, dim3(B * dm.H, (dm.Vd + 15) / 16),
                       dim3(16 * LANES), smem, st, qn, kn, v, coef, state, cu_seqlens, slot_ids, dm, o);
}

template <typename T>
__global__ void delta_output_kernel(const float* __restrict__ o, const T* __restrict__ gate,
                                    int gate_ld, const float* __restrict__ w, float eps,
                                    T* __restrict__ out, int pairs, int H, int Vd) {
  const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  pdl_trigger();
  pdl_wait();
  if (pair >= pairs) return;
  const int t = pair / H, h = pair - t * H;
  const float* src = o + (size_t)pair * Vd;
  float ss = 0.f;
  for (int j = lane; j < Vd; j += 32) ss += src[j] * src[j];
  ss = warp_sum(ss);
  const float rms = sqrtf(ss / (float)Vd + eps);
  for (int j = lane; j < Vd; j += 32) {
    const float gt = sigmoid_f(to_f32(gate[(size_t)t * gate_ld + (size_t)h * Vd + j]));
    out[(size_t)pair * Vd + j] = from_f32<T>(src[j] / rms * w[j] * gt);
  }
}

}  // namespace gf

using namespace gf;
using bf = __nv_bfloat16;

GF_DEFINE_PDL_SWITCH

static DeltaDims dims_of(int H, int G, int D, int Vd, int taps, int state_stride, int conv_off) {
  DeltaDims dm;
  dm.H = H, dm.G = G, dm.D = D, dm.Vd = Vd, dm.taps = taps;
  dm.channels = 2 * G * D + H * Vd;
  dm.state_stride = state_stride, dm.conv_off = conv_off, dm.a_ld = 0;
  return dm;
}

// proj: [T, ld] with the columns q | k | v first and the H beta columns at b_off.
GF_EXPORT int gf_delta_prepare(const void* proj, int ld, int b_off, const float* a,
                               const float* conv_w, const float* dt_bias, const float* A_log,
                               float* state, const int* seq_of_token, const int* cu_seqlens,
                               const int* slot_ids, int T, int B, int H, int G, int D, int Vd,
                               int taps, int state_stride, int conv_off, float* qn, float* kn,
                               float* v, float* g, float* beta, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (H % G || taps < 1) return -3;
  const DeltaDims dm = dims_of(H, G, D, Vd, taps, state_stride, conv_off);
  if (D > 32 * kPrepareMaxPerLane) return -3;
  auto st = (cudaStream_t)stream;
  const int units = 2 * G + 2 * H + 1;
  const dim3 pgrid(T, (units + kPrepareWarps - 1) / kPrepareWarps), pblock(kPrepareWarps * 32);
  int rc;
  if (dtype == GF_F32)
    rc = launch_kernel(delta_prepare_kernel<float, false>, pgrid, pblock, 0, st, (const float*)proj, ld,
                       b_off, a, conv_w, dt_bias, A_log, (const float*)state, seq_of_token,
                       cu_seqlens, slot_ids, dm, qn, kn, v, g, beta);
  else
    rc = launch_kernel(delta_prepare_kernel<bf, false>, pgrid, pblock, 0, st, (const bf*)proj, ld, b_off,
                       a, conv_w, dt_bias, A_log, (const float*)state, seq_of_token, cu_seqlens,
                       slot_ids, dm, qn, kn, v, g, beta);
  if (rc || taps == 1) return rc;
  const dim3 grid((dm.channels + 127) / 128, B);
  if (dtype == GF_F32)
    return launch_kernel(delta_conv_state_kernel<float>, grid, dim3(128), 0, st,
                         (const float*)proj, ld, state, cu_seqlens, slot_ids, dm);
  return launch_kernel(delta_conv_state_kernel<bf>, grid, dim3(128), 0, st, (const bf*)proj, ld,
                       state, cu_seqlens, slot_ids, dm);
}

// One decay a head.  proj: [T, ld] fp32 with the columns q | k | v first and the heads' decay
// pre-activations and betas at a_off and b_off.  max_q_len: the step's longest portion.
GF_EXPORT int gf_delta_prepare_heads(const float* proj, int ld, int a_off, int b_off,
                                     const float* conv_w, const float* dt_bias, const float* A_log,
                                     float* state, const int* seq_of_token, const int* cu_seqlens,
                                     const int* slot_ids, int T, int B, int max_q_len, int H, int G,
                                     int D, int Vd, int taps, int state_stride, int conv_off,
                                     float* qn, float* kn, float* v, float* g, float* beta,
                                     void* stream) {
  if (T <= 0) return 0;
  if (H % G || taps < 1 || D > 32 * kPrepareMaxPerLane) return -3;
  DeltaDims dm = dims_of(H, G, D, Vd, taps, state_stride, conv_off);
  dm.a_ld = ld;
  auto st = (cudaStream_t)stream;
  const int units = 2 * G + H + 1;
  const bool al = (((uintptr_t)proj | (uintptr_t)state | (uintptr_t)qn | (uintptr_t)kn |
                    (uintptr_t)v) & 15) == 0;
  bool updated = false;
  int rc = 1;
  if (D % 4 == 0 && Vd % 4 == 0 && ld % 4 == 0 && state_stride % 4 == 0 && conv_off % 4 == 0 && al &&
      D <= 256 && Vd <= 256 && taps <= 4) {
    // few tokens: one each a warp; many: runs, so that a token's inputs are loaded once
    const int run = T <= 256 ? 1 : 8;
    updated = max_q_len == 1;
    const dim3 grid((T + run - 1) / run, (units + 3) / 4), block(128);
#define GF_GO(TAPS, NQ)                                                                            \
  if (taps == TAPS && D <= 128 * NQ && Vd <= 128 * NQ && rc == 1)                                  \
    rc = launch_kernel(delta_prepare_heads_kernel<TAPS, NQ>, grid, block, 0, st, proj, ld, a_off,  \
                       b_off, conv_w, dt_bias, A_log, state, seq_of_token, cu_seqlens, slot_ids,   \
                       dm, T, run, updated ? 1 : 0, qn, kn, v, g, beta);
    GF_GO(1, 1) GF_GO(2, 1) GF_GO(3, 1) GF_GO(4, 1)
    GF_GO(1, 2) GF_GO(2, 2) GF_GO(3, 2) GF_GO(4, 2)
#undef GF_GO
  } else {
    const dim3 grid(T, (units + kPrepareWarps - 1) / kPrepareWarps), block(kPrepareWarps * 32);
    rc = launch_kernel(delta_prepare_kernel<float, true>, grid, block, 0, st, proj, ld, b_off,
                       proj + a_off, conv_w, dt_bias, A_log, (const float*)state, seq_of_token,
                       cu_seqlens, slot_ids, dm, qn, kn, v, g, beta);
  }
  if (rc || taps == 1 || updated) return rc;
  return launch_kernel(delta_conv_state_kernel<float>, dim3((dm.channels + 127) / 128, B), dim3(128),
                       0, st, proj, ld, state, cu_seqlens, slot_ids, dm);
}

// fp32 words of scratch with which gf_delta_recurrence takes eight tokens at a time (one decay a head).
GF_EXPORT long long gf_delta_chunk_words(int T, int B, int H) {
  return (long long)(T / CT + B + 1) * H * kCoefs;
}

// one_decay: g is [T, H] (a decay a head), else [T, H, D].  scratch (gf_delta_chunk_words; null: token
// by token) and max_q_len, the longest portion, are for steps with one decay a head.
GF_EXPORT int gf_delta_recurrence(const float* qn, const float* kn, const float* v, const float* g,
                                  const float* beta, float* state, const int* cu_seqlens,
                                  const int* slot_ids, int B, int H, int G, int D, int Vd,
                                  int state_stride, float* o, int one_decay, float* scratch,
                                  int max_q_len, void* stream) {
  if (B <= 0) return 0;
  if (H % G) return -3;
  const DeltaDims dm = dims_of(H, G, D, Vd, 1, state_stride, 0);
  auto st = (cudaStream_t)stream;
  if (one_decay && scratch && D % 4 == 0 && Vd % 4 == 0 && D <= 256 && B <= 65535 && G <= 65535 &&
      (((uintptr_t)qn | (uintptr_t)kn | (uintptr_t)v | (uintptr_t)scratch) & 15) == 0) {
    const int chunks = (max_q_len + CT - 1) / CT;
    if (int rc = launch_kernel(delta_chunk_coef_kernel, dim3((chunks + 3) / 4, B, G), dim3(128), 0, st,
                               qn, kn, g, beta, cu_seqlens, dm, scratch))
      return rc;
#define GF_GO(DPER, LANES)                                                                         \
  if (D <= DPER * LANES)                                                                           \
    return launch_chunks<DPER, LANES>(qn, kn, v, scratch, state, cu_seqlens, slot_ids, B, dm, o, st);
    GF_GO(4, 8)
    GF_GO(8, 8)
    GF_GO(16, 8)             // (sixteen lanes of 8 rows: 348 us for a prompt that takes 317 so)
    GF_GO(16, 16)
#undef GF_GO
  }
  // few (request, head, column) triples: a warp (sixteen lanes for key sizes up to 64) a column
  // instead of four lanes (see the kernel)
  const bool wide = (long long)B * H * ((Vd + 31) / 32) < 2 * 148;
  const int lp = !wide ? 4 : (D <= 64 ? 16 : 32);
  const int threads = lp == 32 ? 256 : kRecurrenceThreads;
  const int cols = threads / lp;
  const dim3 grid(B * H, (Vd + cols - 1) / cols);
  const dim3 block(threads);
#define GF_AS(DPER, LP, CHUNK, THREADS, ONE)                                                       \
  {                                                                                                \
    const size_t smem =                                                                            \
        (size_t)kStages * CHUNK * ((ONE ? 2 : 3) * LP * DPER + kMaxColumnsPerBlock + 4) *          \
        sizeof(float);                                                                             \
    return launch_kernel(delta_recurrence_kernel<DPER, LP, CHUNK, THREADS, ONE>, grid, block,      \
                         smem, st, qn, kn, v, g, beta, state, cu_seqlens, slot_ids, dm, o);        \
  }
#define GF_GO(DPER, LP, CHUNK, THREADS)                                                            \
  if (lp == LP && D <= LP * DPER) {                                                                \
    if (one_decay) GF_AS(DPER, LP, CHUNK, THREADS, true)                                           \
    GF_AS(DPER, LP, CHUNK, THREADS, false)                                                         \
  }
  GF_GO(4, 4, 8, kRecurrenceThreads)
  GF_GO(8, 4, 8, kRecurrenceThreads)
  GF_GO(16, 4, 8, kRecurrenceThreads)
  GF_GO(32, 4, 8, kRecurrenceThreads)
  GF_GO(64, 4, 4, kRecurrenceThreads)
  GF_GO(4, 16, 8, kRecurrenceThreads)
  GF_GO(4, 32, 8, 256)
  GF_GO(8, 32, 4, 256)
#undef GF_GO
#undef GF_AS
  return -3;
}

GF_EXPORT int gf_delta_output(const float* o, const void* gate, int gate_ld, const float* w,
                              float eps, void* out, int T, int H, int Vd, int dtype, void* stream) {
  const int pairs = T * H;
  if (pairs <= 0) return 0;
  auto st = (cudaStream_t)stream;
  const dim3 grid((pairs + 3) / 4), block(128);
  if (dtype == GF_F32)
    return launch_kernel(delta_output_kernel<float>, grid, block, 0, st, o, (const float*)gate,
                         gate_ld, w, eps, (float*)out, pairs, H, Vd);
  return launch_kernel(delta_output_kernel<bf>, grid, block, 0, st, o, (const bf*)gate, gate_ld, w,
                       eps, (bf*)out, pairs, H, Vd);
}
