// Shared helpers of the kernel libraries.  Every library is one .cu file built into its own
// shared object with a C ABI: `extern "C" int dinfer_<op>(pointers..., sizes..., cudaStream_t)`.
// A call returns 0, a positive cudaError_t, or a negative refusal code; the text of the last
// refusal or CUDA error of the calling thread is read with dinfer_last_error().
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>
#include <stdio.h>
#include <stdarg.h>
#include <stdlib.h>

#define DINFER_API extern "C" __attribute__((visibility("default")))

enum DinferDtype : int { DINFER_F32 = 0, DINFER_BF16 = 1 };

enum DinferStatus : int {
  DINFER_OK = 0,
  DINFER_BAD_ARGUMENT = -1,   // a size or option the kernel does not take
  DINFER_BAD_DTYPE = -2,
  DINFER_DEVICE_STATUS = -3,  // a kernel recorded a fault in its status word
};

namespace dinfer {

inline char* error_buffer() {
  static thread_local char buf[512] = {0};
  return buf;
}

inline int refuse(int code, const char* fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  vsnprintf(error_buffer(), 512, fmt, ap);
  va_end(ap);
  return code;
}

inline int cuda_status(const char* what) {
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) {
    snprintf(error_buffer(), 512, "%s: %s", what, cudaGetErrorString(e));
    return (int)e;
  }
  return 0;
}

// ---- element types: storage in T, arithmetic in float ----
template <typename T> __device__ __forceinline__ float to_f32(T v);
template <> __device__ __forceinline__ float to_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f32<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

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

// xIELU: quadratic above zero, exponential below, both with the slope 1/2 at zero; a_pos = softplus(p), a_neg = 1/2 +
// softplus(q) of the two numbers that the model learns
__device__ __forceinline__ float xielu(float z, float a_pos, float a_neg) {
  return 0.5f * z + (z > 0.f ? a_pos * z * z : a_neg * (expm1f(z) - z));
}

// The same for results that are rounded to bfloat16, without a branch: e^t - 1 - t by its Taylor polynomial near zero
// (where the difference would cancel), else through the fast exponential.
__device__ __forceinline__ float xielu_fast(float z, float a_pos, float a_neg) {
  const float p = fmaxf(z, 0.f), t = fminf(z, 0.f);
  const float near = t * t * (0.5f + t * (1.f / 6.f + t * (1.f / 24.f + t * (1.f / 120.f + t * (1.f / 720.f)))));
  const float e = t > -0.3f ? near : __expf(t) - 1.f - t;
  return fmaf(0.5f, z, fmaf(a_pos * p, p, a_neg * e));
}

// A gate with a bias on the up side and both sides clamped: g = min(gate, limit), u = clamp(up, -limit, limit),
// g * sigmoid(alpha g) * (u + 1).  `fast`: for results that are rounded to bfloat16.
__device__ __forceinline__ float clamped_swish(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + 1.f);
}
__device__ __forceinline__ float clamped_swish_fast(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g, 1.f + __expf(-alpha * g)) * (u + 1.f);      // 0 where 1 + e^.. passes 2^126, as is its limit
}

// ---- which keys a query sees
// The first key that a query at position pos (>= 0) sees: all of its request's (window <= 0), the last `window` ones
// (itself included), or with `chunked` those of its own chunk (chunks of `window` positions, counted from the
// sequence's first).  It never falls as pos rises.
__device__ __forceinline__ int first_key(int pos, int window, int chunked) {
  if (window <= 0) return 0;
  return chunked ? pos / window * window : max(0, pos - window + 1);
}
// Kept first keys: with keep > 0 a query sees the keys below `keep` too, however far back they lie.  A kernel that walks
// key tiles of BN visits the tiles that hold kept keys and lie before the first tile of its own range [tile_first, ..),
// then its range: `kept_tiles` of them, and visit i is tile `tile_of(i, ...)`.
__device__ __forceinline__ int kept_tiles(int keep, int bn, int tile_first) {
  return min((keep + bn - 1) / bn, tile_first);
}
__device__ __forceinline__ int tile_of(int i, int kept, int tile_first) { return i < kept ? i : tile_first + i - kept; }
// A soft cap on a score, in log2 units: log2(e) * cap * tanh(s / cap) with cap_in = 2 log2(e) / cap (times the score's
// scale) and cap_out = log2(e) * cap.  tanh x = 1 - 2 / (1 + e^2x) through the fast exponential and reciprocal: its error
// is a few 1e-7 of the cap, absolute, which is what a score's error counts by.
__device__ __forceinline__ float softcap_log2(float s, float cap_in, float cap_out) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(s * cap_in));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));       // e = inf gives 0
  return fmaf(-2.f * cap_out, r, cap_out);
}
// The same for four scores with one reciprocal, of the product of the four denominators (the special function unit is what
// such a kernel waits for).  The exponent stops at 30, where tanh has long rounded to 1, so that the product stays finite.
__device__ __forceinline__ void softcap4_log2(float& a, float& b, float& c, float& d, float cap_in, float cap_out) {
  auto denominator = [&](float s) {
    float e;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fminf(s * cap_in, 30.f)));
    return 1.f + e;
  };
  const float da = denominator(a), db = denominator(b), dc = denominator(c), dd = denominator(d);
  const float ab = da * db, cd = dc * dd;
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(ab * cd));
  const float k = -2.f * cap_out * r, rab = k * cd, rcd = k * ab;
  a = fmaf(rab, db, cap_out);
  b = fmaf(rab, da, cap_out);
  c = fmaf(rcd, dd, cap_out);
  d = fmaf(rcd, dc, cap_out);
}
// The softmax's extra term of a head (it has no key and no value): its score times log2(e); the score is sinks[head],
// or 0 where no sinks are given.
__device__ __forceinline__ float sink_log2(const float* sinks, int head) {
  return sinks ? sinks[head] * 1.4426950408889634f : 0.f;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  `scratch` holds 33 floats.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nwarp ? scratch[lane] : 0.f;
    t = warp_sum(t);
    if (lane == 0) scratch[32] = t;
  }
  __syncthreads();
  return scratch[32];
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = (blockDim.x + 31) >> 5;
  v = warp_max(v);
  __syncthreads();
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  if (warp == 0) {
    float t = lane < nwarp ? scratch[lane] : -INFINITY;
    t = warp_max(t);
    if (lane == 0) scratch[32] = t;
  }
  __syncthreads();
  return scratch[32];
}

}  // namespace dinfer

// ---- programmatic dependent launch: a kernel launched through launch_pdl may start while the kernel
// before it on the stream is still running; everything it does before pdl_wait() must be independent
// of all earlier work (no read of their outputs, no write at all).  pdl_wait() returns when the
// preceding kernels have completed and their writes are visible; pdl_launch_dependents() lets the
// NEXT kernel begin its own independent part.  Without the launch attribute both are no-ops.
namespace dinfer {
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
// the usual opening of a kernel with nothing to do ahead of its inputs
__device__ __forceinline__ void pdl_enter() { pdl_launch_dependents(); pdl_wait(); }

// `cluster`: thread-block cluster dimensions (all 1 = no cluster attribute).
template <typename... KArgs, typename... Args>
inline cudaError_t launch_pdl_cluster(void (*kernel)(KArgs...), dim3 grid, dim3 block, dim3 cluster, size_t smem,
                                      cudaStream_t stream, Args... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  unsigned n = 0;
  if (cluster.x * cluster.y * cluster.z > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cluster.x; attr[n].val.clusterDim.y = cluster.y; attr[n].val.clusterDim.z = cluster.z;
    ++n;
  }
  // DINFER_NO_PDL=1 (read once) launches without the attribute: a switch for measuring what the overlap buys
  static const bool off = [] { const char* e = getenv("DINFER_NO_PDL"); return e && e[0] == '1'; }();
  if (!off) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr; cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

template <typename... KArgs, typename... Args>
inline cudaError_t launch_pdl(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                              Args... args) {
  return launch_pdl_cluster(kernel, grid, block, dim3(1, 1, 1), smem, stream, args...);
}
}  // namespace dinfer

// One of these per library gives Python the text of the last refusal.
#define DINFER_DEFINE_LAST_ERROR() \
  DINFER_API const char* dinfer_last_error() { return dinfer::error_buffer(); }

// Call `expr` with T bound to the element type that `code` names.
#define DINFER_DISPATCH_DTYPE(code, T, ...)                                  \
  do {                                                                       \
    if ((code) == DINFER_F32) { using T = float; __VA_ARGS__; }              \
    else if ((code) == DINFER_BF16) { using T = __nv_bfloat16; __VA_ARGS__; }\
    else return dinfer::refuse(DINFER_BAD_DTYPE, "unknown dtype code %d", (int)(code)); \
  } while (0)
