// Shared device helpers: element types, 16-byte vector access, reductions.
//
// Every kernel file of the package is plain CUDA C++ (no torch headers) with
// extern "C" launchers that take raw device pointers and a stream; the Python
// side (redline_b200/ops) loads the shared objects with ctypes.  A launcher
// returns the cudaError_t of its launch as an int (0 = success).
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace rl {

typedef __nv_bfloat16 bf16;

// Number of elements of T in one 16-byte vector.
template <typename T>
struct Vec16 {
  static constexpr int N = 16 / sizeof(T);
};

// Loads one 16-byte vector (address must be 16-byte aligned) into floats.
__device__ __forceinline__ void load16(const float* p, float* out) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  out[0] = v.x; out[1] = v.y; out[2] = v.z; out[3] = v.w;
}
__device__ __forceinline__ void load16(const bf16* p, float* out) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    out[2 * i] = __uint_as_float(w[i] << 16);
    out[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u);
  }
}
__device__ __forceinline__ void store16(float* p, const float* in) {
  *reinterpret_cast<float4*>(p) = make_float4(in[0], in[1], in[2], in[3]);
}
__device__ __forceinline__ void store16(bf16* p, const float* in) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(in[2 * i], in[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&h);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

// Four neighbouring elements as one access (a 16-byte piece of floats, an 8-byte piece of bfloat16).
__device__ __forceinline__ void load4(const float* p, float* out) { load16(p, out); }
__device__ __forceinline__ void load4(const bf16* p, float* out) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  out[0] = __uint_as_float(v.x << 16); out[1] = __uint_as_float(v.x & 0xFFFF0000u);
  out[2] = __uint_as_float(v.y << 16); out[3] = __uint_as_float(v.y & 0xFFFF0000u);
}
__device__ __forceinline__ void store4(float* p, const float* in) { store16(p, in); }
__device__ __forceinline__ void store4(bf16* p, const float* in) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(in[0], in[1]), b = __floats2bfloat162_rn(in[2], in[3]);
  *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

__device__ __forceinline__ float to_float(float x) { return x; }
__device__ __forceinline__ float to_float(bf16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_float(float x);
template <>
__device__ __forceinline__ float from_float<float>(float x) { return x; }
template <>
__device__ __forceinline__ bf16 from_float<bf16>(float x) { return __float2bfloat16_rn(x); }

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

// Sum over the block; `scratch` holds at least 32 floats.  All threads get the result.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();  // scratch may still be read from an earlier call
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float r = (lane < nwarps) ? scratch[lane] : 0.f;
  r = warp_sum(r);
  return r;
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float r = (lane < nwarps) ? scratch[lane] : -INFINITY;
  r = warp_max(r);
  return r;
}

// ---- programmatic dependent launch ----------------------------------------------------
// Kernels of a step form a chain in one stream.  Launched with the programmatic
// stream-serialization attribute, a kernel may begin (be scheduled, run its prologue, ask
// for weights that no earlier kernel writes) while its predecessor is still draining; it
// calls pdl_wait() before it touches anything an earlier kernel of the chain wrote, which
// returns once the predecessor has completed and its writes are visible.  (In a kernel that loads constants before
// pdl_wait(), pointers to what earlier kernels wrote are not `const __restrict__`: loads through such a pointer count
// as loads of memory that never changes, and the compiler may move them up across the wait.)  pdl_launch()
// tells the scheduler that the successor may be brought in.  Without the attribute both
// are no-ops.  REDLINE_PDL=0 in the environment turns the attribute off.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }

}  // namespace rl

#include <cstdlib>
#include <utility>

namespace rl {

inline bool pdl_enabled() {
  static const bool on = [] {
    const char* e = std::getenv("REDLINE_PDL");
    return !(e && e[0] == '0');
  }();
  return on;
}

template <typename... KArgs, typename... Args>
inline cudaError_t launch_kernel(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                 cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

// The same without the attribute: the kernel begins when its predecessor has completed, so its CTAs are
// handed out over an empty machine (a small grid of long-running CTAs that begins while the predecessor drains
// lands on the few SMs that happen to be free first, several CTAs on each, and runs that much longer).
template <typename... KArgs, typename... Args>
inline cudaError_t launch_kernel_serial(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                                        cudaStream_t stream, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cfg.attrs = nullptr;
  cfg.numAttrs = 0;
  return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

}  // namespace rl

#define RL_LAUNCH_END() return static_cast<int>(cudaGetLastError())
