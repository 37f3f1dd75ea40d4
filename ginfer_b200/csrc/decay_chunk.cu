// The linear recurrence with ONE decay a head and token over long portions, a chunk of kC tokens at a
// time (decay_state.cu has the recurrence itself, token after token):
//
//     S_t = g_t S_(t-1) + c_t k_t v_t^T,   o_t = S_t^T q_t (+ skip_h v_t),   n_t = g_t n_(t-1) + c_t k_t
//
// With R[t, j] = c_j prod_(j < i <= t) g_i and G_t = prod_(i <= t) g_i inside a chunk that starts from S:
//
//     o_t = sum_(j <= t) R[t, j] (q_t . k_j) v_j + G_t S^T q_t,    S' = G_end S + sum_j R[end, j] k_j v_j^T
//
//   decay_chunk_state_kernel  a block a (chunk, head, tile of S): the chunk's own part of S' (and of n').
//   decay_chunk_scan_kernel   a thread four elements of a request's state: walks over its chunks, leaves
//                             every chunk the state it starts from, and brings the slot up to date.
//   decay_chunk_out_kernel    a block a (chunk, head, tile of columns): the scores q . k, weighted by R,
//                             times v, and the part of the state the chunk starts from.
//
// Ratios of decays are products of the factors between two tokens, never quotients, so a decay of zero or
// one loses nothing.  All products are fp32 multiply-adds: the state and what enters it are 32-bit.
#include "common.cuh"

namespace gf {

constexpr int kC = 64;             // tokens a chunk
constexpr int kSlab = 32;          // rows of S, channels of K a stage
constexpr int kThreads = 256;      // 16 x 16, a thread 4 rows x 4 NV columns
constexpr int kMaxSeqs = 1024;

struct ChunkDims {
  int H, G, D, Vd, B;
  int ld_q, ld_k, ld_v, ld_g, ld_c, ld_o, ld_n;
  int state_stride, norm_off;      // norm_off < 0: no normaliser
};

struct ChunkPlace {
  int b, row0, len;                // request, first row of the step's tokens, tokens
};

// Chunk number -> its place; every thread gets it.  cu: [B + 1].  False past the last chunk.
__device__ __forceinline__ bool find_chunk(int chunk, const int* cu, int B, int* scratch,
                                           ChunkPlace& at) {
  if (threadIdx.x < 32) {
    int before = 0, found = -1, base = 0;
    for (int b0 = 0; b0 < B && found < 0; b0 += 32) {
      const int b = b0 + threadIdx.x;
      const int n = b < B ? (cu[b + 1] - cu[b] + kC - 1) / kC : 0;
      int incl = n;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, incl, o);
        if ((int)threadIdx.x >= o) incl += up;
      }
      const bool mine = chunk < before + incl && chunk >= before + incl - n;
      const unsigned hit = __ballot_sync(0xffffffffu, mine);
      if (hit) {
        const int src = __ffs(hit) - 1;
        found = b0 + src;
        base = __shfl_sync(0xffffffffu, before + incl - n, src);
      }
      before += __shfl_sync(0xffffffffu, incl, 31);
    }
    if (threadIdx.x == 0) scratch[0] = found, scratch[1] = base;
  }
  __syncthreads();
  at.b = scratch[0];
  if (at.b < 0) return false;
  const int first = cu[at.b] + (chunk - scratch[1]) * kC;
  at.row0 = first;
  at.len = min(kC, cu[at.b + 1] - first);
  return true;
}

// acc[4][4 NV] += a (4 rows) x b (4 NV columns), columns 4 tx .. + 3 of every 64
template <int NV>
__device__ __forceinline__ void outer(float (&acc)[4][4 * NV], const float* a, const float* b, int tx) {
  const float4 av = *reinterpret_cast<const float4*>(a);
  const float ar[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
  for (int n = 0; n < NV; ++n) {
    const float4 bv = *reinterpret_cast<const float4*>(b + 64 * n + 4 * tx);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      acc[i][4 * n] = fmaf(ar[i], bv.x, acc[i][4 * n]);
      acc[i][4 * n + 1] = fmaf(ar[i], bv.y, acc[i][4 * n + 1]);
      acc[i][4 * n + 2] = fmaf(ar[i], bv.z, acc[i][4 * n + 2]);
      acc[i][4 * n + 3] = fmaf(ar[i], bv.w, acc[i][4 * n + 3]);
    }
  }
}

// grid (chunks, H, D tiles of 64 x column tiles of 64 NV)
template <int NV>
__global__ void __launch_bounds__(kThreads)
decay_chunk_state_kernel(const float* __restrict__ k, const float* __restrict__ v,
                         const float* __restrict__ g, const float* __restrict__ c,
                         const int* __restrict__ cu_seqlens, ChunkDims dm, float* __restrict__ parts,
                         float* __restrict__ nparts, float* __restrict__ gains) {
  constexpr int BV = 64 * NV;
  extern __shared__ __align__(16) float sm[];
  float* ks = sm;                          // [kC][64], times R[end, j]
  float* vs = sm + kC * 64;                // [kC][BV]
  __shared__ float gs[kC], rs[kC];
  __shared__ int where[2];
  const int chunk = blockIdx.x, h = blockIdx.y;
  const int vtiles = (dm.Vd + BV - 1) / BV;
  const int d0 = (blockIdx.z / vtiles) * 64, v0 = (blockIdx.z % vtiles) * BV;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  pdl_trigger();
  pdl_wait();
  ChunkPlace at;
  if (!find_chunk(chunk, cu_seqlens, dm.B, where, at)) return;
  const int gk = h / (dm.H / dm.G);
  if (threadIdx.x < kC) {
    const bool in = threadIdx.x < at.len;
    const size_t r = (size_t)(at.row0 + threadIdx.x);
    gs[threadIdx.x] = in ? g[r * dm.ld_g + h] : 1.f;
    rs[threadIdx.x] = in ? (c ? c[r * dm.ld_c + h] : 1.f) : 0.f;
  }
  for (int i = threadIdx.x; i < kC * BV / 4; i += kThreads) {
    const int j = i / (BV / 4), col = (i - j * (BV / 4)) * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < at.len && v0 + col < dm.Vd)
      x = *reinterpret_cast<const float4*>(v + (size_t)(at.row0 + j) * dm.ld_v + (size_t)h * dm.Vd + v0 + col);
    *reinterpret_cast<float4*>(vs + j * BV + col) = x;
  }
  __syncthreads();
  if (threadIdx.x < kC) {                  // R[end, j]: the factors behind token j
    float r = rs[threadIdx.x];
    for (int i = kC - 1; i > (int)threadIdx.x; --i) r *= gs[i];
    rs[threadIdx.x] = r;
  } else if (threadIdx.x == kC && blockIdx.z == 0) {
    float all = 1.f;
    for (int i = 0; i < kC; ++i) all *= gs[i];
    gains[(size_t)chunk * dm.H + h] = all;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kC * 16; i += kThreads) {
    const int j = i >> 4, d = (i & 15) * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < at.len && d0 + d < dm.D) {
      x = *reinterpret_cast<const float4*>(k + (size_t)(at.row0 + j) * dm.ld_k + (size_t)gk * dm.D + d0 + d);
      const float r = rs[j];
      x.x *= r, x.y *= r, x.z *= r, x.w *= r;
    }
    *reinterpret_cast<float4*>(ks + j * 64 + d) = x;
  }
  __syncthreads();
  float acc[4][4 * NV] = {};
  for (int j = 0; j < at.len; ++j) outer<NV>(acc, ks + j * 64 + 4 * ty, vs + j * BV, tx);
  float* dst = parts + ((size_t)chunk * dm.H + h) * dm.D * dm.Vd;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int d = d0 + 4 * ty + i;
    if (d >= dm.D) continue;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int col = v0 + 64 * n + 4 * tx;
      if (col < dm.Vd)
        *reinterpret_cast<float4*>(dst + (size_t)d * dm.Vd + col) =
            make_float4(acc[i][4 * n], acc[i][4 * n + 1], acc[i][4 * n + 2], acc[i][4 * n + 3]);
    }
  }
  if (nparts != nullptr && v0 == 0 && threadIdx.x < 64 && d0 + threadIdx.x < dm.D) {
    float s = 0.f;
    for (int j = 0; j < at.len; ++j) s += ks[j * 64 + threadIdx.x];
    nparts[((size_t)chunk * dm.H + h) * dm.D + d0 + threadIdx.x] = s;
  }
}

// grid (quads of a head's state and normaliser / 256, H, B)
__global__ void __launch_bounds__(256)
decay_chunk_scan_kernel(float* __restrict__ parts, float* __restrict__ nparts,
                        const float* __restrict__ gains, float* __restrict__ state,
                        const int* __restrict__ cu_seqlens, const int* __restrict__ slot_ids,
                        ChunkDims dm) {
  const int h = blockIdx.y, b = blockIdx.z;
  const int quads = dm.D * dm.Vd / 4, nq = dm.norm_off >= 0 ? dm.D / 4 : 0;
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  pdl_trigger();
  pdl_wait();
  if (e >= quads + nq) return;
  int first = 0;
  for (int i = 0; i < b; ++i) first += (cu_seqlens[i + 1] - cu_seqlens[i] + kC - 1) / kC;
  const int count = (cu_seqlens[b + 1] - cu_seqlens[b] + kC - 1) / kC;
  const bool isn = e >= quads;
  const int el = isn ? e - quads : e;
  const size_t size = isn ? dm.D / 4 : quads;                       // quads between two heads
  float4* p = reinterpret_cast<float4*>(isn ? nparts : parts) + ((size_t)first * dm.H + h) * size + el;
  float* slot = state + (size_t)slot_ids[b] * dm.state_stride +
                (isn ? (size_t)dm.norm_off + (size_t)h * dm.D : (size_t)h * dm.D * dm.Vd) + 4 * el;
  float s[4] = {slot[0], slot[1], slot[2], slot[3]};                // (a slot need not be 16-byte aligned)
  const float* gain = gains + (size_t)first * dm.H + h;
  const size_t step = (size_t)dm.H * size;
  constexpr int U = 8;                                              // chunks whose loads go out together
  for (int c0 = 0; c0 < count; c0 += U) {
    float4 u[U];
    float gn[U];
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (c0 + i < count) u[i] = p[(c0 + i) * step], gn[i] = gain[(size_t)(c0 + i) * dm.H];
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (c0 + i < count) {
        p[(c0 + i) * step] = make_float4(s[0], s[1], s[2], s[3]);
        s[0] = fmaf(gn[i], s[0], u[i].x);
        s[1] = fmaf(gn[i], s[1], u[i].y);
        s[2] = fmaf(gn[i], s[2], u[i].z);
        s[3] = fmaf(gn[i], s[3], u[i].w);
      }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) slot[i] = s[i];
}

// Shared memory of the read-out: q^T [Dp][kC], R and later its weighted scores transposed, and a stage
// that holds in turn a slab of k^T, slabs of S, and v.
__host__ __device__ constexpr int padded_keys(int D) { return (D + kSlab - 1) / kSlab * kSlab; }
__host__ __device__ constexpr int out_floats(int D, int BV) {
  return padded_keys(D) * kC + kC * (kC + 1) + kC * kC + kC * BV;
}

// grid (chunks, H, column tiles of 64 NV)
template <int NV>
__global__ void __launch_bounds__(kThreads)
decay_chunk_out_kernel(const float* __restrict__ q, const float* __restrict__ k,
                       const float* __restrict__ v, const float* __restrict__ g,
                       const float* __restrict__ c, const float* __restrict__ skip,
                       const int* __restrict__ cu_seqlens, ChunkDims dm,
                       const float* __restrict__ starts, const float* __restrict__ nstarts,
                       float* __restrict__ o, float* __restrict__ o_norm) {
  constexpr int BV = 64 * NV;
  extern __shared__ __align__(16) float sm[];
  const int D = dm.D, Dp = padded_keys(D);
  float* qt = sm;                          // [Dp][kC]
  float* R = qt + Dp * kC;                 // [kC][kC + 1]
  float* mt = R + kC * (kC + 1);           // [kC][kC]: weighted scores, mt[j][t]  (16-byte aligned: kC
  float* stage = mt + kC * kC;             //  (kC + 1) is a multiple of four)
  __shared__ float gs[kC], cs[kC], Gt[kC], nsum[kC];
  __shared__ int where[2];
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * BV;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, warp = threadIdx.x >> 5;
  pdl_trigger();
  pdl_wait();
  ChunkPlace at;
  if (!find_chunk(chunk, cu_seqlens, dm.B, where, at)) return;
  const int gk = h / (dm.H / dm.G);
  const int lt = threadIdx.x & (kC - 1), lq = threadIdx.x >> 6;      // loads: a token, one of 4 quads
  auto transposed = [&](float* dst, const float* src, int ld, int d0, int width) {
    for (int e = lq * 4; e < width; e += 16) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (lt < at.len && d0 + e < D)
        x = *reinterpret_cast<const float4*>(src + (size_t)(at.row0 + lt) * ld + (size_t)gk * D + d0 + e);
      dst[e * kC + lt] = x.x;
      dst[(e + 1) * kC + lt] = x.y;
      dst[(e + 2) * kC + lt] = x.z;
      dst[(e + 3) * kC + lt] = x.w;
    }
  };
  if (threadIdx.x < kC) {
    const bool in = threadIdx.x < at.len;
    const size_t r = (size_t)(at.row0 + threadIdx.x);
    gs[threadIdx.x] = in ? g[r * dm.ld_g + h] : 0.f;
    cs[threadIdx.x] = in ? (c ? c[r * dm.ld_c + h] : 1.f) : 0.f;
  }
  transposed(qt, q, dm.ld_q, 0, Dp);
  __syncthreads();
  if (threadIdx.x < kC) {                  // column j of R
    const int j = threadIdx.x;
    float r = cs[j];
    for (int t = 0; t < kC; ++t) {
      if (t > j) r *= gs[t];
      R[t * (kC + 1) + j] = t >= j ? r : 0.f;
    }
  } else if (threadIdx.x == kC) {
    float all = 1.f;
    for (int t = 0; t < kC; ++t) Gt[t] = all *= gs[t];
  }
  // scores: P = Q K^T, a thread 4 tokens x 4 keys
  float sc[4][4] = {};
  for (int d0 = 0; d0 < Dp; d0 += kSlab) {
    __syncthreads();                       // the stage is free (and, at first, R is there)
    transposed(stage, k, dm.ld_k, d0, kSlab);
    __syncthreads();
#pragma unroll 8
    for (int d = 0; d < kSlab; ++d) outer<1>(sc, qt + (d0 + d) * kC + 4 * ty, stage + d * kC, tx);
  }
  float rowsum[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    rowsum[i] = 0.f;
#pragma unroll
    for (int jj = 0; jj < 4; ++jj) {
      sc[i][jj] *= R[(4 * ty + i) * (kC + 1) + 4 * tx + jj];
      rowsum[i] += sc[i][jj];
    }
#pragma unroll
    for (int off = 1; off < 16; off <<= 1) rowsum[i] += __shfl_xor_sync(0xffffffffu, rowsum[i], off);
    if (tx == 0) nsum[4 * ty + i] = rowsum[i];
  }
#pragma unroll
  for (int jj = 0; jj < 4; ++jj)
    *reinterpret_cast<float4*>(mt + (4 * tx + jj) * kC + 4 * ty) =
        make_float4(sc[0][jj], sc[1][jj], sc[2][jj], sc[3][jj]);
  // the state the chunk starts from: acc = Q S, then row t times G_t
  float acc[4][4 * NV] = {};
  const float* S = starts + ((size_t)chunk * dm.H + h) * D * dm.Vd;
  for (int d0 = 0; d0 < Dp; d0 += kSlab) {
    __syncthreads();
    for (int i = threadIdx.x; i < kSlab * BV / 4; i += kThreads) {
      const int d = i / (BV / 4), col = (i - d * (BV / 4)) * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d0 + d < D && v0 + col < dm.Vd)
        x = *reinterpret_cast<const float4*>(S + (size_t)(d0 + d) * dm.Vd + v0 + col);
      *reinterpret_cast<float4*>(stage + d * BV + col) = x;
    }
    __syncthreads();
#pragma unroll 8
    for (int d = 0; d < kSlab; ++d) outer<NV>(acc, qt + (d0 + d) * kC + 4 * ty, stage + d * BV, tx);
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float gt = Gt[4 * ty + i];
#pragma unroll
    for (int n = 0; n < 4 * NV; ++n) acc[i][n] *= gt;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kC * BV / 4; i += kThreads) {
    const int j = i / (BV / 4), col = (i - j * (BV / 4)) * 4;
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (j < at.len && v0 + col < dm.Vd)
      x = *reinterpret_cast<const float4*>(v + (size_t)(at.row0 + j) * dm.ld_v + (size_t)h * dm.Vd + v0 + col);
    *reinterpret_cast<float4*>(stage + j * BV + col) = x;
  }
  __syncthreads();
  // a warp's eight tokens see keys up to the last of them
  const int keys = min(at.len, 8 * warp + 8);
  for (int j = 0; j < keys; ++j) outer<NV>(acc, mt + j * kC + 4 * ty, stage + j * BV, tx);
  const float sk = skip != nullptr ? skip[h] : 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = 4 * ty + i;
    if (t >= at.len) continue;
    float* dst = o + (size_t)(at.row0 + t) * dm.ld_o + (size_t)h * dm.Vd + v0;
#pragma unroll
    for (int n = 0; n < NV; ++n) {
      const int col = 64 * n + 4 * tx;
      if (v0 + col >= dm.Vd) continue;
      const float* vv = stage + t * BV + col;
      *reinterpret_cast<float4*>(dst + col) =
          make_float4(fmaf(sk, vv[0], acc[i][4 * n]), fmaf(sk, vv[1], acc[i][4 * n + 1]),
                      fmaf(sk, vv[2], acc[i][4 * n + 2]), fmaf(sk, vv[3], acc[i][4 * n + 3]));
    }
  }
  if (o_norm != nullptr && blockIdx.z == 0 && threadIdx.x < at.len) {
    const float* n0 = nstarts + ((size_t)chunk * dm.H + h) * D;
    float s = 0.f;
    for (int d = 0; d < D; ++d) s = fmaf(qt[d * kC + threadIdx.x], n0[d], s);
    o_norm[(size_t)(at.row0 + threadIdx.x) * dm.ld_n + h] = fmaf(Gt[threadIdx.x], s, nsum[threadIdx.x]);
  }
}

}  // namespace gf

using namespace gf;

GF_DEFINE_PDL_SWITCH

GF_EXPORT int gf_decay_chunk_tokens() { return kC; }

// Arguments as gf_decay_recurrence has them, with one decay a head; `chunks`: the sum over the requests of
// their tokens over gf_decay_chunk_tokens(), rounded up.  scratch: chunks * H * (D * Vd + D + 1) floats.
// -6: not served (key sizes over 128, sizes, strides or pointers that are no multiple of four elements).
GF_EXPORT int gf_decay_chunked(const float* q, int ld_q, const float* k, int ld_k, const float* v, int ld_v,
                               const float* g, int ld_g, const float* c, int ld_c, const float* skip,
                               float* state, int state_stride, const int* cu_seqlens, const int* slot_ids,
                               int B, int chunks, int H, int G, int D, int Vd, float* o, int ld_o,
                               int norm_off, float* o_norm, int ld_n, float* scratch, void* stream) {
  if (B <= 0 || chunks <= 0) return 0;
  auto aligned = [](const void* p, int ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; };
  if (G <= 0 || H % G || D <= 0 || D > 128 || D % 4 || Vd <= 0 || Vd % 4 || B > kMaxSeqs || H > 65535 ||
      !aligned(q, ld_q) || !aligned(k, ld_k) || !aligned(v, ld_v) || !aligned(o, ld_o) ||
      !aligned(scratch, 0) || (o_norm && norm_off < 0))
    return -6;
  ChunkDims dm;
  dm.H = H, dm.G = G, dm.D = D, dm.Vd = Vd, dm.B = B;
  dm.ld_q = ld_q, dm.ld_k = ld_k, dm.ld_v = ld_v, dm.ld_g = ld_g, dm.ld_c = ld_c, dm.ld_o = ld_o;
  dm.ld_n = ld_n, dm.state_stride = state_stride, dm.norm_off = o_norm ? norm_off : -1;
  float* parts = scratch;
  float* nparts = parts + (size_t)chunks * H * D * Vd;
  float* gains = nparts + (size_t)chunks * H * D;
  auto st = (cudaStream_t)stream;
  const int nv = Vd > 64 ? 2 : 1, BV = 64 * nv, vtiles = (Vd + BV - 1) / BV, dtiles = (D + 63) / 64;
  const size_t smem_s = (size_t)(kC * 64 + kC * BV) * sizeof(float);
  const size_t smem_o = (size_t)out_floats(D, BV) * sizeof(float);
  const dim3 sgrid(chunks, H, dtiles * vtiles), ogrid(chunks, H, vtiles), block(kThreads);
  const int quads = D * Vd / 4 + (o_norm ? D / 4 : 0);
  const dim3 cgrid((quads + 255) / 256, H, B);
#define GF_GO(NV)                                                                                     \
  {                                                                                                   \
    static OncePerDevice attrs;                                                                       \
    if (int rc = attrs.run([&] {                                                                      \
          cudaError_t e = cudaFuncSetAttribute(decay_chunk_state_kernel<NV>,                          \
                                               cudaFuncAttributeMaxDynamicSharedMemorySize,           \
                                               (kC * 64 + kC * 64 * NV) * (int)sizeof(float));        \
          if (e != cudaSuccess) return e;                                                             \
          return cudaFuncSetAttribute(decay_chunk_out_kernel<NV>,                                     \
                                      cudaFuncAttributeMaxDynamicSharedMemorySize,                    \
                                      out_floats(128, 64 * NV) * (int)sizeof(float));                 \
        }))                                                                                           \
      return rc;                                                                                      \
    int rc = launch_kernel(decay_chunk_state_kernel<NV>, sgrid, block, smem_s, st, k, v, g, c,        \
                           cu_seqlens, dm, parts, o_norm ? nparts : (float*)nullptr, gains);          \
    if (rc) return rc;                                                                                \
    rc = launch_kernel(decay_chunk_scan_kernel, cgrid, dim3(256), 0, st, parts, nparts,               \
                       (const float*)gains, state, cu_seqlens, slot_ids, dm);                         \
    if (rc) return rc;                                                                                \
    return launch_kernel(decay_chunk_out_kernel<NV>, ogrid, block, smem_o, st, q, k, v, g, c, skip,   \
                         cu_seqlens, dm, (const float*)parts, (const float*)nparts, o, o_norm);       \
  }
  if (nv == 2) GF_GO(2)
  GF_GO(1)
#undef GF_GO
}
