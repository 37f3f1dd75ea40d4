// Rotation by position of the heads of a projection that leaves its product in 32-bit:
//
//   rotary_heads_kernel   q and k heads rotated in place (fp32), k times a constant: the operands of a
//                         linear attention with positions.
//   rotary_write_kernel   q | k | v with their biases, q and k rotated; q leaves in the activation
//                         type, k and v go to their cache slots.  Heads may be stored wider than they
//                         are (zero channels behind the true ones) for attention kernels that take
//                         certain head sizes only.
//
// Pairs are neighbours (2i, 2i + 1) or halves (i, i + n); the angle is float(position) * freqs[i] in
// fp32, its sine and cosine are taken once a token, into shared memory.  Channels from 2 n on pass.
#include "common.cuh"

namespace gf {

struct RotaryDims {
  int nq, nk, D;            // q heads, k heads, channels of a head
  int q_off, k_off;         // columns of a row where they start
  int n_pairs, neighbours;
};

__device__ __forceinline__ void angle_table(float* tab, int n_pairs, const float* freqs, float pos) {
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x)
    sincosf(pos * freqs[i], &tab[n_pairs + i], &tab[i]);
}

// A block a token; a thread a pair (or a channel behind the rotated ones) of a head at a time.
__global__ void rotary_heads_kernel(float* __restrict__ p, int ld, const RotaryDims dm,
                                    const float* __restrict__ freqs, float k_scale,
                                    const int* __restrict__ positions, int early) {
  extern __shared__ __align__(16) float tab[];        // cos[n], sin[n]
  const int t = blockIdx.x, n = dm.n_pairs, D = dm.D;
  if (early) pdl_trigger();
  pdl_wait();
  angle_table(tab, n, freqs, (float)positions[t]);
  __syncthreads();
  float* row = p + (size_t)t * ld;
  const int per = D - n;                              // pairs, then the channels behind them
  const int total = (dm.nq + dm.nk) * per;
  for (int it = threadIdx.x; it < total; it += blockDim.x) {
    const int h = it / per, e = it - h * per;
    const bool is_k = h >= dm.nq;
    if (!is_k && e >= n) continue;                    // q's other channels stay as they are
    float* x = row + (is_k ? dm.k_off + (h - dm.nq) * D : dm.q_off + h * D);
    const float f = is_k ? k_scale : 1.f;
    if (e < n) {
      const int a = dm.neighbours ? 2 * e : e, b = dm.neighbours ? 2 * e + 1 : e + n;
      const float u = x[a], v = x[b], cs = tab[e], sn = tab[n + e];
      x[a] = (u * cs - v * sn) * f;
      x[b] = (v * cs + u * sn) * f;
    } else {
      x[n + e] *= f;
    }
  }
}

// The same for halves with D and n multiples of 4 and 16-byte aligned heads, four channels an access.
__global__ void rotary_heads_vec_kernel(float* __restrict__ p, int ld, const RotaryDims dm,
                                        const float* __restrict__ freqs, float k_scale,
                                        const int* __restrict__ positions, int early) {
  extern __shared__ __align__(16) float tab[];
  const int t = blockIdx.x, n = dm.n_pairs, D = dm.D;
  if (early) pdl_trigger();
  pdl_wait();
  angle_table(tab, n, freqs, (float)positions[t]);
  __syncthreads();
  float* row = p + (size_t)t * ld;
  const int nq4 = n >> 2, per = (D - n) >> 2;
  const int total = (dm.nq + dm.nk) * per;
  for (int it = threadIdx.x; it < total; it += blockDim.x) {
    const int h = it / per, e = it - h * per;
    const bool is_k = h >= dm.nq;
    if (!is_k && e >= nq4) continue;
    float* x = row + (is_k ? dm.k_off + (h - dm.nq) * D : dm.q_off + h * D);
    const float f = is_k ? k_scale : 1.f;
    if (e < nq4) {
      float u[4], v[4], cs[4], sn[4];
      Quad<float>::load(x + 4 * e, u);
      Quad<float>::load(x + n + 4 * e, v);
      Quad<float>::load(tab + 4 * e, cs);
      Quad<float>::load(tab + n + 4 * e, sn);
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = (u[i] * cs[i] - v[i] * sn[i]) * f;
        b[i] = (v[i] * cs[i] + u[i] * sn[i]) * f;
      }
      Quad<float>::store(x + 4 * e, a);
      Quad<float>::store(x + n + 4 * e, b);
    } else {
      float u[4];
      Quad<float>::load(x + n + 4 * e, u);
#pragma unroll
      for (int i = 0; i < 4; ++i) u[i] *= f;
      Quad<float>::store(x + n + 4 * e, u);
    }
  }
}

struct RotaryWriteDims {
  int nh, nkv, hd, vd;      // heads; true channels of a key and of a value head
  int kd, kv;               // stored channels of a q / k head and of a value head
  int q_off, k_off, v_off;  // columns of a projection row
  int n_pairs, neighbours;
};

// A block a token, a thread an output channel at a time.
template <typename T>
__global__ void rotary_write_kernel(const float* __restrict__ p, int ld, const RotaryWriteDims dm,
                                    const float* __restrict__ bias,
                                    const float* __restrict__ freqs,
                                    const int* __restrict__ positions,
                                    const int* __restrict__ slot_mapping, T* __restrict__ q,
                                    T* __restrict__ kpages, T* __restrict__ vpages) {
  extern __shared__ __align__(16) float tab[];
  const int t = blockIdx.x, n = dm.n_pairs;
  pdl_trigger();
  pdl_wait();
  angle_table(tab, n, freqs, (float)positions[t]);
  __syncthreads();
  const float* row = p + (size_t)t * ld;
  const size_t slot = slot_mapping ? (size_t)slot_mapping[t] : 0;
  auto at = [&](int col) { return row[col] + (bias ? bias[col] : 0.f); };
  const int nq = dm.nh * dm.kd, nk = slot_mapping ? dm.nkv * dm.kd : 0;
  const int nv = slot_mapping ? dm.nkv * dm.kv : 0;
  for (int i = threadIdx.x; i < nq + nk + nv; i += blockDim.x) {
    if (i >= nq + nk) {
      const int e = i - nq - nk, h = e / dm.kv, c = e - h * dm.kv;
      vpages[slot * nv + e] = from_f32<T>(c < dm.vd ? at(dm.v_off + h * dm.vd + c) : 0.f);
      continue;
    }
    const bool is_k = i >= nq;
    const int e = is_k ? i - nq : i, h = e / dm.kd, c = e - h * dm.kd;
    const int base = (is_k ? dm.k_off : dm.q_off) + h * dm.hd;
    float y = 0.f;
    if (c < 2 * n) {
      const bool second = dm.neighbours ? (c & 1) : c >= n;
      const int pair = dm.neighbours ? c >> 1 : (second ? c - n : c);
      const int other = dm.neighbours ? (c ^ 1) : (second ? c - n : c + n);
      const float me = at(base + c), ot = at(base + other);
      y = second ? me * tab[pair] + ot * tab[n + pair] : me * tab[pair] - ot * tab[n + pair];
    } else if (c < dm.hd) {
      y = at(base + c);
    }
    if (is_k) kpages[slot * nk + e] = from_f32<T>(y);
    else q[(size_t)t * nq + e] = from_f32<T>(y);
  }
}

// The same for neighbours, four channels an access: all sizes and offsets multiples of four, pointers
// aligned to four elements.
template <typename T>
__global__ void rotary_write_vec_kernel(const float* __restrict__ p, int ld,
                                        const RotaryWriteDims dm, const float* __restrict__ bias,
                                        const float* __restrict__ freqs,
                                        const int* __restrict__ positions,
                                        const int* __restrict__ slot_mapping, T* __restrict__ q,
                                        T* __restrict__ kpages, T* __restrict__ vpages) {
  extern __shared__ __align__(16) float tab[];
  const int t = blockIdx.x, n = dm.n_pairs;
  pdl_trigger();
  pdl_wait();
  angle_table(tab, n, freqs, (float)positions[t]);
  __syncthreads();
  const float* row = p + (size_t)t * ld;
  const size_t slot = slot_mapping ? (size_t)slot_mapping[t] : 0;
  const int kq = dm.kd >> 2, vq = dm.kv >> 2;
  const int nq = dm.nh * kq, nk = slot_mapping ? dm.nkv * kq : 0, nv = slot_mapping ? dm.nkv * vq : 0;
  for (int i = threadIdx.x; i < nq + nk + nv; i += blockDim.x) {
    const bool is_v = i >= nq + nk, is_k = !is_v && i >= nq;
    const int e = is_v ? i - nq - nk : is_k ? i - nq : i;
    const int per = is_v ? vq : kq, h = e / per, c = 4 * (e - h * per);
    const int size = is_v ? dm.vd : dm.hd;
    const int col = (is_v ? dm.v_off : is_k ? dm.k_off : dm.q_off) + h * size + c;
    float x[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < size) {
      Quad<float>::load(row + col, x);
      if (bias) {
        float b[4];
        Quad<float>::load(bias + col, b);
#pragma unroll
        for (int j = 0; j < 4; ++j) x[j] += b[j];
      }
      if (!is_v) {
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          const int pair = (c + j) >> 1;
          if (pair < n) {
            const float u = x[j], v = x[j + 1], cs = tab[pair], sn = tab[n + pair];
            x[j] = u * cs - v * sn;
            x[j + 1] = v * cs + u * sn;
          }
        }
      }
    }
    T* dst = is_v ? vpages + (slot * nv + e) * 4
                  : is_k ? kpages + (slot * nk + e) * 4 : q + ((size_t)t * nq + e) * 4;
    Quad<T>::store(dst, x);
  }
}

}  // namespace gf

using namespace gf;
using bf = __nv_bfloat16;

GF_DEFINE_PDL_SWITCH

// p: [T, ld] fp32.  freqs [n_pairs] (null with n_pairs 0).  early: whether the kernel behind this one
// may start before this grid has drained.
GF_EXPORT int gf_rotary_heads(float* p, int ld, int T, int nq, int nk, int D, int q_off, int k_off,
                              const float* freqs, int n_pairs, int neighbours, float k_scale,
                              const int* positions, int early, void* stream) {
  if (T <= 0) return 0;
  if (n_pairs < 0 || 2 * n_pairs > D || (n_pairs > 0 && !freqs)) return -3;
  const RotaryDims dm{nq, nk, D, q_off, k_off, n_pairs, neighbours};
  auto st = (cudaStream_t)stream;
  const size_t smem = 2 * (size_t)n_pairs * sizeof(float);
  const bool vec = !neighbours && n_pairs % 4 == 0 && D % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 &&
                   k_off % 4 == 0 && ((uintptr_t)p & 15) == 0;
  const int items = (nq + nk) * (D - n_pairs) / (vec ? 4 : 1);
  const dim3 grid(T), block(items >= 512 ? 512 : items > 128 ? 256 : 128);
  if (vec)
    return launch_kernel(rotary_heads_vec_kernel, grid, block, smem, st, p, ld, dm, freqs, k_scale,
                         positions, early);
  return launch_kernel(rotary_heads_kernel, grid, block, smem, st, p, ld, dm, freqs, k_scale,
                       positions, early);
}

// p: [T, ld] fp32 rows; bias: fp32, one a column of p, or null.  q: [T, nh, kd]; kpages [.., nkv, kd],
// vpages [.., nkv, kv]; slot_mapping null: nothing is cached.
GF_EXPORT int gf_rotary_write(const float* p, int ld, int T, int nh, int nkv, int hd, int vd, int kd,
                              int kv, int q_off, int k_off, int v_off, const float* bias,
                              const float* freqs, int n_pairs, int neighbours,
                              const int* positions, const int* slot_mapping, void* q, void* kpages,
                              void* vpages, int dtype, void* stream) {
  if (T <= 0) return 0;
  if (n_pairs < 0 || 2 * n_pairs > hd || (n_pairs > 0 && !freqs) || kd < hd || kv < vd) return -3;
  const RotaryWriteDims dm{nh, nkv, hd, vd, kd, kv, q_off, k_off, v_off, n_pairs, neighbours};
  auto st = (cudaStream_t)stream;
  const size_t smem = 2 * (size_t)n_pairs * sizeof(float), es = dtype == GF_F32 ? 4 : 2;
  const bool vec = (neighbours || n_pairs == 0) &&
                   (hd | vd | kd | kv | q_off | k_off | v_off | ld) % 4 == 0 &&
                   ((uintptr_t)p & 15) == 0 && ((uintptr_t)bias & 15) == 0 &&
                   (((uintptr_t)q | (uintptr_t)kpages | (uintptr_t)vpages) % (4 * es)) == 0;
  const int items = (nh * kd + nkv * (kd + kv)) / (vec ? 4 : 1);
  const dim3 grid(T), block(items >= 512 ? 512 : items > 128 ? 256 : 128);
#define GF_GO(K, TT)                                                                                \
  return launch_kernel(K<TT>, grid, block, smem, st, p, ld, dm, bias, freqs, positions,             \
                       slot_mapping, (TT*)q, (TT*)kpages, (TT*)vpages)
  if (vec) {
    if (dtype == GF_F32) GF_GO(rotary_write_vec_kernel, float);
    GF_GO(rotary_write_vec_kernel, bf);
  }
  if (dtype == GF_F32) GF_GO(rotary_write_kernel, float);
  GF_GO(rotary_write_kernel, bf);
#undef GF_GO
}
