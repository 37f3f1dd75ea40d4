// Shared device helpers for the hand-written sm_100a kernels.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <mutex>

#define GF_EXPORT extern "C" __attribute__((visibility("default")))

// dtype codes used across the C interface
#define GF_F32 0
#define GF_BF16 1

namespace gf {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return (uint32_t)__cvta_generic_to_shared(p);
}

// xIELU: a z^2 + z/2 above zero, b (e^z - 1 - z) + z/2 below.  Close to zero e^z - 1 - z comes from
// its power series (six terms: relative error below 1e-6 down to -1/4), where the difference would
// lose its digits.
__device__ __forceinline__ float xielu(float z, float a, float b) {
  const float z2 = z * z;
  const float series =
      z2 * fmaf(z, fmaf(z, fmaf(z, fmaf(z, 1.f / 720.f, 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f);
  const float below = z > -0.25f ? series : __expf(z) - 1.f - z;
  return fmaf(0.5f, z, z > 0.f ? a * z2 : b * below);
}

template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) {
  return __bfloat162float(v);
}
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) {
  return __float2bfloat16_rn(v);
}

// Four channels of one type as one access (the address a multiple of four elements).
template <typename T> struct Quad;
template <> struct Quad<float> {
  static __device__ __forceinline__ void load(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
};
template <> struct Quad<__nv_bfloat16> {
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
    const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
    v[0] = a.x, v[1] = a.y, v[2] = b.x, v[3] = b.y;
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&v)[4]) {
    uint2 raw;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
    h[0] = __floats2bfloat162_rn(v[0], v[1]);
    h[1] = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = raw;
  }
};

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();                      // scratch may still be read from an earlier call
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nwarps ? scratch[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) scratch[32] = t;
  }
  __syncthreads();
  return scratch[32];
}

inline int launch_status() { return (int)cudaGetLastError(); }

// The first key the query at position p sees (the last one is p itself).  `span` is how the
// attention kernels are told their mask: 0 = every earlier key; span > 0 = a sliding window of
// `span` keys (p - c < span); span < 0 = chunks of -span positions counted from position 0 of the
// sequence (a query sees the keys of its own chunk).  Never decreases with p.
__host__ __device__ __forceinline__ int first_visible_key(int p, int span) {
  if (span > 0) return p - span + 1 > 0 ? p - span + 1 : 0;
  if (span < 0) return p / (-span) * (-span);
  return 0;
}

// Shaped attention scores.  With a cap, score <- cap * tanh(score / cap) after the scale; with
// slopes (one a head), slope * (p - c) is then taken off the score of the key at c for the query at
// p.  A sink adds exp(sink) to the softmax's denominator: a key with this score and no value.
// 32-bit arithmetic in every kernel that takes it.
constexpr float kNoSink = -__builtin_inff();
// The sink's score: one for all heads (kNoSink: none), or one a head.
struct Sink {
  float score;
  const float* heads;     // [heads], or null: `score` is every head's
  __device__ __forceinline__ float at(int head) const { return heads ? heads[head] : score; }
};
struct ScoreShape {
  float cap;              // 0: no cap
  const float* slopes;    // [heads], or null: no distance bias
  Sink sink;
};
// Whether single scores change (the sink only enters a row's sum, at its end).
__host__ __device__ __forceinline__ bool shaped(const ScoreShape& sh) {
  return sh.cap > 0.f || sh.slopes != nullptr;
}
// What a sink adds to a row's sum of 2^(score - m) when everything is in log2 units; nothing for
// kNoSink.  m is the row's reference maximum (finite: a query sees itself).
__device__ __forceinline__ float sink_share(float sink, float m_log2) {
  return exp2f(fmaf(sink, 1.4426950408889634f, -m_log2));
}

// ---- programmatic dependent launch -------------------------------------------------------------
// A kernel launched with the attribute may start while its predecessor in the stream still runs;
// it must call pdl_wait() before it reads (or overwrites) anything the predecessor touches, and
// may do independent work first (set-up, loading weights).  pdl_trigger() lets the successor start.
// Launched without the attribute, both are no-ops.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_trigger() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

// An index that a kernel shortly before this one wrote, read from L2.  A kernel that was launched while
// that one still ran may share its SM with kernels that read the same memory when it held something
// else (a recycled buffer), and what they left in L1 must not be taken for an index.
__device__ __forceinline__ int fresh_index(const int* p) { return __ldcg(p); }

inline int& pdl_flag() {
  static int enabled = 1;
  return enabled;
}

// cluster > 1 launches thread-block clusters of (1, 1, cluster), or (cluster, 1, 1) with along_x.
template <typename... KArgs, typename... Args>
inline int launch_kernel_cluster_dims(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                      cudaStream_t stream, int cluster_z, bool along_x,
                                      Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (pdl_flag()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  if (cluster_z > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = along_x ? (unsigned)cluster_z : 1;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = along_x ? 1 : (unsigned)cluster_z;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  return (int)cudaLaunchKernelEx(&cfg, kernel, KArgs(args)...);
}

template <typename... KArgs, typename... Args>
inline int launch_kernel_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                 cudaStream_t stream, int cluster_z, Args... args) {
  return launch_kernel_cluster_dims(kernel, grid, block, smem, stream, cluster_z, false, args...);
}

template <typename... KArgs, typename... Args>
inline int launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                         cudaStream_t stream, Args... args) {
  return launch_kernel_cluster_dims(kernel, grid, block, smem, stream, 1, false, args...);
}

}  // namespace gf

// Every library exports this switch for programmatic dependent launch (on by default).
// A kernel's attributes (dynamic shared memory, cluster sizes) belong to a device: `set` runs once
// on each device a launcher is used on.  Returns `set`'s error, -9 for a device that cannot be
// told, else 0.  One object per launcher and attribute set (a function-local static).
struct OncePerDevice {
  static constexpr int kMaxDevices = 64;
  std::mutex lock;
  bool done[kMaxDevices] = {};
  template <typename F>
  int run(F&& set) {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= kMaxDevices) return -9;
    std::lock_guard<std::mutex> hold(lock);
    if (done[dev]) return 0;
    const cudaError_t e = set();
    if (e != cudaSuccess) return (int)e;
    done[dev] = true;
    return 0;
  }
};

#define GF_DEFINE_PDL_SWITCH \
  GF_EXPORT void gf_set_pdl(int on) { gf::pdl_flag() = on ? 1 : 0; }
