// The start of a sublayer that reads a token-shifted norm, together with the end of the sublayer in
// front of it, on a 32-bit residual stream over packed tokens of several requests:
//
//   v_t = x_t + y_t * gamma_b / rms(y_t)      (y null: v = x)
//   n_t = v_t * gamma / rms(v_t)
//   h_t = n_t + (n_(t-1) - n_t) * w           (w a weight a channel)
//
// n_(t-1) is the row of the token before in the same request: the row above, or, for the first token
// of a portion, what the request's state slot holds (n of the last token of earlier steps, zero at
// the start).  v leaves in fp32, h in the activation type; n itself is never rounded.
//
// A row's n is formed again by whoever needs it as a neighbour.  The slot: whoever owns a portion's
// FIRST row reads it, and the same threads form the portion's LAST n and write that to the slot
// afterwards, so no other block's reads can meet the write.
#include "common.cuh"

namespace gf {

struct ShiftArgs {
  const float* x;            // [T, H]
  const void* y;             // [T, H] or null
  const float* gamma_b;
  float eps_b;
  float* out;                // [T, H] (null: not wanted)
  const float* gamma;
  float eps;
  const float* w;
  float* state;              // [slots, H]
  const int* seq_of_token;
  const int* cu_seqlens;
  const int* slot_ids;
  void* h;                   // [T, H]
  int T, H;
};

// Any row length: a block a row, rows in shared memory.
template <typename Y>
__device__ __forceinline__ void form_row(const ShiftArgs& a, int r, float* row, float* scratch,
                                         bool store) {
  const size_t base = (size_t)r * a.H;
  float scale = 0.f;
  if (a.y) {
    const Y* y = reinterpret_cast<const Y*>(a.y);
    float ss = 0.f;
    for (int j = threadIdx.x; j < a.H; j += blockDim.x) {
      const float v = to_f32(y[base + j]);
      ss += v * v;
    }
    scale = sqrtf(block_sum(ss, scratch) / (float)a.H + a.eps_b);
  }
  float s2 = 0.f;
  for (int j = threadIdx.x; j < a.H; j += blockDim.x) {
    float v = a.x[base + j];
    if (a.y) v += to_f32(reinterpret_cast<const Y*>(a.y)[base + j]) * a.gamma_b[j] / scale;
    if (store && a.out) a.out[base + j] = v;
    row[j] = v;
    s2 += v * v;
  }
  const float rms = sqrtf(block_sum(s2, scratch) / (float)a.H + a.eps);
  for (int j = threadIdx.x; j < a.H; j += blockDim.x) row[j] = row[j] / rms * a.gamma[j];
}

template <typename Y, typename T>
__global__ void norm_shift_kernel(const ShiftArgs a) {
  extern __shared__ __align__(16) float rows[];      // n of this row | n of the row before
  __shared__ float scratch[33];
  const int r = blockIdx.x;
  pdl_trigger();
  pdl_wait();
  const int b = a.seq_of_token[r], start = a.cu_seqlens[b], last = a.cu_seqlens[b + 1] - 1;
  float* slot = a.state + (size_t)a.slot_ids[b] * a.H;
  float *mine = rows, *before = rows + a.H;
  form_row<Y>(a, r, mine, scratch, true);
  if (r == start) {
    for (int j = threadIdx.x; j < a.H; j += blockDim.x) before[j] = slot[j];
  } else {
    form_row<Y>(a, r - 1, before, scratch, false);
  }
  T* h = reinterpret_cast<T*>(a.h) + (size_t)r * a.H;
  for (int j = threadIdx.x; j < a.H; j += blockDim.x)      // a thread reads what it wrote itself
    h[j] = from_f32<T>(mine[j] + (before[j] - mine[j]) * a.w[j]);
  if (r != start) return;
  if (last != r) form_row<Y>(a, last, mine, scratch, false);
  for (int j = threadIdx.x; j < a.H; j += blockDim.x) slot[j] = mine[j];
}

// Four channels an access, rows in registers.  blockDim = (threads a row, row groups).  HALO: group 0
// holds the row in front of the block's first one, the others a row each, and a row's n reaches the
// group behind it through shared memory.  Without HALO (every portion of the step is one token) a
// block is one row.
template <int OPT>
constexpr int shift_threads() { return OPT <= 4 ? 1024 : 512; }

template <typename Y, typename T, int OPT, bool HALO>
__global__ void __launch_bounds__(shift_threads<OPT>())
norm_shift_vec_kernel(const ShiftArgs a) {
  extern __shared__ __align__(16) float rows[];      // HALO: n of every group's row
  __shared__ float scratch[2][32];
  const int nq = a.H >> 2, group = HALO ? threadIdx.y : 0;
  const int warps = blockDim.x >> 5, wid = threadIdx.x >> 5;
  const int r = HALO ? (int)blockIdx.x * ((int)blockDim.y - 1) + group - 1 : (int)blockIdx.x;
  pdl_trigger();
  float gb[OPT][4];
  if (!HALO && a.y) {                                // weights: before the wait
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (q < nq) Quad<float>::load(a.gamma_b + 4 * q, gb[u]);
    }
  }
  pdl_wait();
  const bool live = r >= 0 && r < a.T;
  const int b = live ? a.seq_of_token[r] : 0;
  const int start = live ? a.cu_seqlens[b] : 0, last = live ? a.cu_seqlens[b + 1] - 1 : 0;
  float* slot = a.state + (live ? (size_t)a.slot_ids[b] * a.H : 0);

  // sum over the threads of a group; every thread of the block comes here
  auto row_sum = [&](float v, int which) {
    v = warp_sum(v);
    if (warps == 1) return v;
    if ((threadIdx.x & 31) == 0) scratch[which][group * warps + wid] = v;
    __syncthreads();
    float s = 0.f;
    for (int i = 0; i < warps; ++i) s += scratch[which][group * warps + i];
    return s;
  };
  float n[OPT][4];
  // n of row rr into registers (nothing of the block's barriers depends on rr)
  auto form = [&](int rr, bool ok, bool store) {
    const size_t base = (size_t)(ok ? rr : 0) * a.H;
    float inv_b = 0.f;
    if (a.y) {
      const Y* y = reinterpret_cast<const Y*>(a.y);
      float ss = 0.f;
#pragma unroll
      for (int u = 0; u < OPT; ++u) {
        const int q = threadIdx.x + u * blockDim.x;
        if (ok && q < nq) {
          Quad<Y>::load(y + base + 4 * q, n[u]);
#pragma unroll
          for (int i = 0; i < 4; ++i) ss += n[u][i] * n[u][i];
        }
      }
      inv_b = 1.f / sqrtf(row_sum(ss, 0) / (float)a.H + a.eps_b);
    }
    float s2 = 0.f;
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (ok && q < nq) {
        float xv[4];
        Quad<float>::load(a.x + base + 4 * q, xv);
        if (a.y) {
          float g4[4];
          if (HALO) Quad<float>::load(a.gamma_b + 4 * q, g4);
#pragma unroll
          for (int i = 0; i < 4; ++i) n[u][i] = xv[i] + n[u][i] * (HALO ? g4[i] : gb[u][i]) * inv_b;
        } else {
#pragma unroll
          for (int i = 0; i < 4; ++i) n[u][i] = xv[i];
        }
        if (store && a.out) Quad<float>::store(a.out + base + 4 * q, n[u]);
#pragma unroll
        for (int i = 0; i < 4; ++i) s2 += n[u][i] * n[u][i];
      }
    }
    const float inv = 1.f / sqrtf(row_sum(s2, 1) / (float)a.H + a.eps);
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (ok && q < nq) {
        float g4[4];
        Quad<float>::load(a.gamma + 4 * q, g4);
#pragma unroll
        for (int i = 0; i < 4; ++i) n[u][i] = n[u][i] * inv * g4[i];
      }
    }
  };
  const bool mine = live && (!HALO || group > 0);     // a row of this block's own
  form(r, live, mine);
  if (HALO) {
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (live && q < nq) Quad<float>::store(rows + (size_t)group * a.H + 4 * q, n[u]);
    }
    __syncthreads();
  }
  const bool first = mine && r == start;
  if (mine) {
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (q < nq) {
        float p[4], w4[4], o[4];
        if (HALO && !first) Quad<float>::load(rows + (size_t)(group - 1) * a.H + 4 * q, p);
        else Quad<float>::load(slot + 4 * q, p);
        Quad<float>::load(a.w + 4 * q, w4);
#pragma unroll
        for (int i = 0; i < 4; ++i) o[i] = n[u][i] + (p[i] - n[u][i]) * w4[i];
        Quad<T>::store(reinterpret_cast<T*>(a.h) + (size_t)r * a.H + 4 * q, o);
      }
    }
  }
  if (HALO) {                                         // a portion's last n, where its first row lives
    const bool again = first && last != r;
    if (__syncthreads_or(again)) form(last, again, false);
  }
  if (first) {
#pragma unroll
    for (int u = 0; u < OPT; ++u) {
      const int q = threadIdx.x + u * blockDim.x;
      if (q < nq) Quad<float>::store(slot + 4 * q, n[u]);
    }
  }
}

template <typename Y, typename T, int OPT>
static int launch_vec(const ShiftArgs& a, bool single, int per_row, cudaStream_t st) {
  if (single)
    return launch_kernel(norm_shift_vec_kernel<Y, T, OPT, false>, dim3(a.T), dim3(per_row), 0, st, a);
  // as many row groups as the block's threads, its sums (32 warps) and 96 KB of shared memory allow
  int groups = shift_threads<OPT>() / per_row;
  if (groups > 8) groups = 8;
  const int fit = (int)((96 * 1024) / ((size_t)a.H * sizeof(float)));
  if (groups > fit) groups = fit;
  if (groups < 2) return -4;
  const size_t smem = (size_t)groups * a.H * sizeof(float);
  static OncePerDevice attrs;
  if (int rc = attrs.run([&] {
        return cudaFuncSetAttribute(norm_shift_vec_kernel<Y, T, OPT, true>,
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);
      }))
    return rc;
  return launch_kernel(norm_shift_vec_kernel<Y, T, OPT, true>,
                       dim3((a.T + groups - 2) / (groups - 1)), dim3(per_row, groups), smem, st, a);
}

}  // namespace gf

using namespace gf;
using bf = __nv_bfloat16;

GF_DEFINE_PDL_SWITCH

// x [T, H] fp32, y [T, H] in y_dtype or null (gamma_b, eps_b: the norm it passes), out (nullable)
// [T, H] fp32, gamma / eps: the norm in front, w [H], state [slots, H]; h [T, H] in act_dtype.
// max_q_len: the longest portion of the step.  -4: rows too long for shared memory.
GF_EXPORT int gf_norm_shift(const float* x, const void* y, int y_dtype, const float* gamma_b,
                            float eps_b, float* out, const float* gamma, float eps, const float* w,
                            float* state, const int* seq_of_token, const int* cu_seqlens,
                            const int* slot_ids, void* h, int act_dtype, int T, int H, int max_q_len,
                            void* stream) {
  if (T <= 0) return 0;
  if (y && act_dtype == GF_F32 && y_dtype != GF_F32) return -2;
  auto st = (cudaStream_t)stream;
  const ShiftArgs a{x, y, gamma_b, eps_b, out, gamma, eps, w, state, seq_of_token, cu_seqlens,
                    slot_ids, h, T, H};
  const bool al = (((uintptr_t)x | (uintptr_t)y | (uintptr_t)gamma_b | (uintptr_t)out |
                    (uintptr_t)gamma | (uintptr_t)w | (uintptr_t)state | (uintptr_t)h) & 15) == 0;
  const bool single = max_q_len == 1;
  if (H % 4 == 0 && al && H <= 4 * 8 * 256) {
    const int nq = H / 4;
    // threads a row: more where a row has the SM to itself (single tokens)
    int per_row = single ? 256 : nq <= 4 * 128 ? 128 : nq <= 8 * 128 ? 128 : 256;
    if (nq <= 32) per_row = 32;
    else if (nq <= 64 && !single) per_row = 64;
    else if (nq <= 128 && single) per_row = 128;
    const int opt = (nq + per_row - 1) / per_row;
#define GF_OPT(Y, T)                                                       \
  {                                                                        \
    if (opt <= 1) return launch_vec<Y, T, 1>(a, single, per_row, st);      \
    if (opt <= 2) return launch_vec<Y, T, 2>(a, single, per_row, st);      \
    if (opt <= 4) return launch_vec<Y, T, 4>(a, single, per_row, st);      \
    return launch_vec<Y, T, 8>(a, single, per_row, st);                    \
  }
    if (act_dtype == GF_F32) GF_OPT(float, float)
    if (!y || y_dtype == GF_F32) GF_OPT(float, bf)
    GF_OPT(bf, bf)
#undef GF_OPT
  }
  const size_t smem = 2 * (size_t)H * sizeof(float);
  if (smem > 48 * 1024) return -4;
  const dim3 grid(T), block(H >= 512 ? 256 : 128);
  if (act_dtype == GF_F32) return launch_kernel(norm_shift_kernel<float, float>, grid, block, smem, st, a);
  if (!y || y_dtype == GF_F32)
    return launch_kernel(norm_shift_kernel<float, bf>, grid, block, smem, st, a);
  return launch_kernel(norm_shift_kernel<bf, bf>, grid, block, smem, st, a);
}
