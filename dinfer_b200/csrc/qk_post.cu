// After the q/k/v projection, in one pass over a token's heads: per-head RMSNorm of q and k,
// neox rotation of the first `rot` dims by the angle table row of the token's position, q and k
// written back in place, and k and v written to the token's slot of the paged cache.
// Every piece is optional (null weight / null table / null cache), so the same kernel serves a
// mixer without head norm, without rotation, or one that reads another layer's cache.
//
// Cache layout, per layer: [num_blocks, 2 (k, v), Hkv, block_size, D]; slot = block*block_size + offset.
// Counterpart in the reference: crates/kernels/cuda/qkv_post.cu:26-91 (D in {128, 256} only there).
#include "common.cuh"

using namespace dinfer;

namespace {

constexpr int WARPS = 8;
constexpr int MAX_D = 512;

// eight consecutive elements at once
template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 x = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
#pragma unroll
  for (int j = 0; j < 4; ++j) { const float2 f = __bfloat1622float2(h[j]); v[2 * j] = f.x; v[2 * j + 1] = f.y; }
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  uint4 x;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&x);
#pragma unroll
  for (int j = 0; j < 4; ++j) h[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
  *reinterpret_cast<uint4*>(p) = x;
}

// One warp per (token, head); a lane owns runs of 8 elements (VEC8) or single elements.
template <typename TA, typename TW, bool VEC8>
__global__ void __launch_bounds__(WARPS * 32)
qk_post_kernel(TA* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
               const TW* __restrict__ q_weight, const TW* __restrict__ k_weight, float eps,
               const float* __restrict__ cos_sin, int rot, int interleaved,
               TA* __restrict__ cache, const int* __restrict__ slots, int block_size,
               int H, int Hkv, int D) {
  __shared__ __align__(16) float sm[WARPS][MAX_D];
  pdl_enter();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * WARPS + warp;
  if (head >= H + 2 * Hkv) return;
  const int kind = head < H ? 0 : (head < H + Hkv ? 1 : 2);   // q, k, v
  TA* x = qkv + (int64_t)t * ld + (int64_t)head * D;
  float* xs = sm[warp];
  constexpr int STEP = VEC8 ? 8 : 1;

  const TW* w = kind == 0 ? q_weight : (kind == 1 ? k_weight : nullptr);
  float ss = 0.f;
  for (int e = lane * STEP; e < D; e += 32 * STEP) {
    if (VEC8) {
      float v[8];
      load8<TA>(x + e, v);
#pragma unroll
      for (int j = 0; j < 8; ++j) { xs[e + j] = v[j]; ss += v[j] * v[j]; }
    } else {
      const float v = to_f32<TA>(x[e]);
      xs[e] = v;
      ss += v * v;
    }
  }
  if (w) {
    ss = warp_sum(ss);
    const float rinv = rsqrtf(ss / (float)D + eps);
    for (int e = lane * STEP; e < D; e += 32 * STEP) {
#pragma unroll
      for (int j = 0; j < STEP; ++j) xs[e + j] = xs[e + j] * rinv * to_f32<TW>(w[e + j]);
    }
  }
  __syncwarp();

  TA* dst = nullptr;
  if (cache && kind != 0) {
    const int slot = slots[t];
    if (slot >= 0) {
      const int64_t blk = slot / block_size, off = slot % block_size;
      const int hk = kind == 1 ? head - H : head - H - Hkv;
      dst = cache + ((((blk * 2 + (kind - 1)) * Hkv + hk) * block_size + off) * (int64_t)D);
    }
  }
  const bool rotate = cos_sin != nullptr && kind != 2;
  const bool rewrite = kind != 2 && (w || rotate);
  const int half = rot >> 1;
  const float* cs = rotate ? cos_sin + (int64_t)positions[t] * rot : nullptr;
  for (int e0 = lane * STEP; e0 < D; e0 += 32 * STEP) {
    float r[8];
#pragma unroll
    for (int j = 0; j < STEP; ++j) {
      const int e = e0 + j;
      float v = xs[e];
      if (rotate && e < rot) {
        if (interleaved) {                                    // pairs (2i, 2i + 1), angle i
          const int i = e >> 1;
          v = (e & 1) ? v * cs[i] + xs[e - 1] * cs[half + i] : v * cs[i] - xs[e + 1] * cs[half + i];
        } else if (e < half) {                                // pairs (i, i + rot/2), angle i
          v = v * cs[e] - xs[e + half] * cs[half + e];
        } else {
          v = v * cs[e - half] + xs[e - half] * cs[e];
        }
      }
      r[j] = v;
    }
    if (VEC8) {
      if (rewrite) store8<TA>(x + e0, r);
      if (dst) store8<TA>(dst + e0, r);
    } else {
      const TA o = from_f32<TA>(r[0]);
      if (rewrite) x[e0] = o;
      if (dst) dst[e0] = o;
    }
  }
}

// Fast shape: bfloat16/f32 with D = 32 * EPL and the rotation over the whole head.  A lane owns EPL
// consecutive elements in registers; its rotation partner (D/2 away) sits 16 lanes across.  A warp takes
// HPW consecutive heads of one token and requests all of them before it works on the first, so that
// enough bytes are in flight for prompts (one 8-byte load per lane and head is not).
constexpr int HPW = 4;

template <typename TA, typename TW, int EPL>
__global__ void __launch_bounds__(WARPS * 32)
qk_post_lanes_kernel(TA* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
                     const TW* __restrict__ q_weight, const TW* __restrict__ k_weight, float eps,
                     const float* __restrict__ cos_sin, TA* __restrict__ cache, const int* __restrict__ slots,
                     int block_size, int H, int Hkv) {
  constexpr int D = 32 * EPL;
  struct alignas(sizeof(TA) * EPL) Vec { TA v[EPL]; };
  struct alignas(sizeof(TW) * EPL) WVec { TW v[EPL]; };
  struct alignas(sizeof(float) * EPL) FVec { float v[EPL]; };
  pdl_enter();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head0 = (blockIdx.y * WARPS + warp) * HPW;
  const int heads = H + 2 * Hkv;
  if (head0 >= heads) return;
  TA* row = qkv + (int64_t)t * ld + lane * EPL;
  Vec in[HPW];
#pragma unroll
  for (int u = 0; u < HPW; ++u)
    if (head0 + u < heads) in[u] = *reinterpret_cast<const Vec*>(row + (int64_t)(head0 + u) * D);
  FVec c, sn;
  const bool has_table = cos_sin != nullptr;
  if (has_table) {
    const float* cs = cos_sin + (int64_t)positions[t] * D;
    const int i = (lane & 15) * EPL;                          // index of the pair inside the half
    c = *reinterpret_cast<const FVec*>(cs + i);
    sn = *reinterpret_cast<const FVec*>(cs + D / 2 + i);
  }
  const int slot = cache ? slots[t] : -1;
#pragma unroll
  for (int u = 0; u < HPW; ++u) {
    const int head = head0 + u;
    if (head >= heads) break;
    const int kind = head < H ? 0 : (head < H + Hkv ? 1 : 2);
    float v[EPL];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < EPL; ++j) { v[j] = to_f32<TA>(in[u].v[j]); ss += v[j] * v[j]; }
    const TW* w = kind == 0 ? q_weight : (kind == 1 ? k_weight : nullptr);
    if (w) {
      ss = warp_sum(ss);
      const float rinv = rsqrtf(ss / (float)D + eps);
      const WVec wv = *reinterpret_cast<const WVec*>(w + lane * EPL);
#pragma unroll
      for (int j = 0; j < EPL; ++j) v[j] = v[j] * rinv * to_f32<TW>(wv.v[j]);
    }
    const bool rotate = has_table && kind != 2;
    if (rotate) {
#pragma unroll
      for (int j = 0; j < EPL; ++j) {
        const float other = __shfl_xor_sync(0xffffffffu, v[j], 16);
        v[j] = lane < 16 ? v[j] * c.v[j] - other * sn.v[j] : v[j] * c.v[j] + other * sn.v[j];
      }
    }
    Vec out;
#pragma unroll
    for (int j = 0; j < EPL; ++j) out.v[j] = from_f32<TA>(v[j]);
    if (kind != 2 && (w || rotate)) *reinterpret_cast<Vec*>(row + (int64_t)head * D) = out;
    if (kind != 0 && slot >= 0) {
      const int64_t blk = slot / block_size, off = slot % block_size;
      const int hk = kind == 1 ? head - H : head - H - Hkv;
      TA* dst = cache + ((((blk * 2 + (kind - 1)) * Hkv + hk) * block_size + off) * (int64_t)D) + lane * EPL;
      *reinterpret_cast<Vec*>(dst) = out;
    }
  }
}

// Head size 128 in bfloat16, the rotation over the whole head: half a warp per head.  A lane owns four consecutive
// elements of the head's first half and the four elements 64 further on, which are their rotation partners, so the
// rotation needs no exchange between lanes (two 8-byte accesses a head).  A warp takes HALF_HP pairs of heads (one
// where the tokens are few: a decode step is a chain of latencies, more warps make it shorter) of one
// token and requests all of them before it works on the first.  Value heads are only copied into the cache.
constexpr int FEW_TOKENS = 128;

__device__ __forceinline__ void unpack4(const uint2& x, float (&v)[4]) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&x);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ uint2 pack4(const float (&v)[4]) {
  uint2 x;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&x);
  h[0] = __floats2bfloat162_rn(v[0], v[1]);
  h[1] = __floats2bfloat162_rn(v[2], v[3]);
  return x;
}

template <typename TW, int HALF_HP>
__global__ void __launch_bounds__(WARPS * 32)
qk_post_half_warp_kernel(__nv_bfloat16* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
                         const TW* __restrict__ q_weight, const TW* __restrict__ k_weight, float eps,
                         const float* __restrict__ cos_sin, __nv_bfloat16* __restrict__ cache,
                         const int* __restrict__ slots, int block_size, int H, int Hkv) {
  constexpr int D = 128;
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int side = lane >> 4, l = lane & 15;
  const int head0 = (blockIdx.y * WARPS + warp) * 2 * HALF_HP + side;
  const int heads = H + 2 * Hkv;
  // What no kernel of the step writes (the token's position and slot, its row of the angle table, the norm weights)
  // is fetched while the kernel before this one may still be running; the q/k/v rows only after it has completed.
  pdl_launch_dependents();
  float4 c = make_float4(1.f, 1.f, 1.f, 1.f), sn = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool has_table = cos_sin != nullptr;
  if (has_table) {
    const float* cs = cos_sin + (int64_t)positions[t] * D + l * 4;
    c = *reinterpret_cast<const float4*>(cs);
    sn = *reinterpret_cast<const float4*>(cs + D / 2);
  }
  const float cv[4] = {c.x, c.y, c.z, c.w}, sv[4] = {sn.x, sn.y, sn.z, sn.w};
  const int slot = cache ? slots[t] : -1;
  const int64_t blk = slot >= 0 ? slot / block_size : 0, off = slot >= 0 ? slot % block_size : 0;
  float wq[2][4], wk[2][4];                                    // this lane's norm weights: [half of the head][element]
  auto weights = [&](const TW* w, float (&dst)[2][4]) {
    if (!w) {
#pragma unroll
      for (int j = 0; j < 4; ++j) dst[0][j] = dst[1][j] = 1.f;
    } else if constexpr (sizeof(TW) == 2) {
      unpack4(*reinterpret_cast<const uint2*>(w + l * 4), dst[0]);
      unpack4(*reinterpret_cast<const uint2*>(w + D / 2 + l * 4), dst[1]);
    } else {
      const float4 x = *reinterpret_cast<const float4*>(w + l * 4), y = *reinterpret_cast<const float4*>(w + D / 2 + l * 4);
      dst[0][0] = x.x; dst[0][1] = x.y; dst[0][2] = x.z; dst[0][3] = x.w;
      dst[1][0] = y.x; dst[1][1] = y.y; dst[1][2] = y.z; dst[1][3] = y.w;
    }
  };
  weights(q_weight, wq);
  weights(k_weight, wk);
  pdl_wait();
  __nv_bfloat16* row = qkv + (int64_t)t * ld + l * 4;          // this lane's elements of the first half
  uint2 lo[HALF_HP], hi[HALF_HP];
#pragma unroll
  for (int u = 0; u < HALF_HP; ++u)
    if (head0 + 2 * u < heads) {
      lo[u] = *reinterpret_cast<const uint2*>(row + (int64_t)(head0 + 2 * u) * D);
      hi[u] = *reinterpret_cast<const uint2*>(row + (int64_t)(head0 + 2 * u) * D + D / 2);
    }
#pragma unroll
  for (int u = 0; u < HALF_HP; ++u) {
    const int head = head0 + 2 * u;
    const bool live = head < heads;                            // (the other half of the warp may still have a head)
    const int kind = head < H ? 0 : (head < H + Hkv ? 1 : 2);
    const TW* w = !live ? nullptr : (kind == 0 ? q_weight : (kind == 1 ? k_weight : nullptr));
    const bool rotate = has_table && live && kind != 2;
    uint2 out_lo = lo[u], out_hi = hi[u];
    float a[4], b[4];
    float ss = 0.f;
    if (live && kind != 2) {
      unpack4(lo[u], a);
      unpack4(hi[u], b);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += a[j] * a[j] + b[j] * b[j];
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);     // over the head's 16 lanes
    if (live && kind != 2) {
      if (w) {
        const float rinv = rsqrtf(ss / (float)D + eps);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          a[j] = a[j] * rinv * (kind == 0 ? wq[0][j] : wk[0][j]);
          b[j] = b[j] * rinv * (kind == 0 ? wq[1][j] : wk[1][j]);
        }
      }
      if (rotate) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float x = a[j], y = b[j];
          a[j] = x * cv[j] - y * sv[j];
          b[j] = y * cv[j] + x * sv[j];
        }
      }
      out_lo = pack4(a);
      out_hi = pack4(b);
      if (w || rotate) {
        *reinterpret_cast<uint2*>(row + (int64_t)head * D) = out_lo;
        *reinterpret_cast<uint2*>(row + (int64_t)head * D + D / 2) = out_hi;
      }
    }
    if (live && kind != 0 && slot >= 0) {
      const int hk = kind == 1 ? head - H : head - H - Hkv;
      __nv_bfloat16* dst = cache + ((((blk * 2 + (kind - 1)) * Hkv + hk) * block_size + off) * (int64_t)D) + l * 4;
      *reinterpret_cast<uint2*>(dst) = out_lo;
      *reinterpret_cast<uint2*>(dst + D / 2) = out_hi;
    }
  }
}

template <typename TA, typename TW>
void launch_lanes(dim3 grid, cudaStream_t stream, TA* qkv, int64_t ld, const int* positions, const TW* qw,
                  const TW* kw, float eps, const float* cos_sin, TA* cache, const int* slots, int block_size,
                  int H, int Hkv, int D) {
  const int threads = WARPS * 32;
  if (D == 32) launch_pdl(qk_post_lanes_kernel<TA, TW, 1>, grid, dim3(threads), 0, stream, qkv, ld, positions, qw, kw, eps, cos_sin, cache, slots, block_size, H, Hkv);
  else if (D == 64) launch_pdl(qk_post_lanes_kernel<TA, TW, 2>, grid, dim3(threads), 0, stream, qkv, ld, positions, qw, kw, eps, cos_sin, cache, slots, block_size, H, Hkv);
  else if (D == 128) launch_pdl(qk_post_lanes_kernel<TA, TW, 4>, grid, dim3(threads), 0, stream, qkv, ld, positions, qw, kw, eps, cos_sin, cache, slots, block_size, H, Hkv);
  else launch_pdl(qk_post_lanes_kernel<TA, TW, 8>, grid, dim3(threads), 0, stream, qkv, ld, positions, qw, kw, eps, cos_sin, cache, slots, block_size, H, Hkv);
}

}  // namespace

DINFER_DEFINE_LAST_ERROR()

// qkv [T, >= (H+2Hkv)*D] act dtype with row stride ld, laid out q heads | k heads | v heads.
// positions [T] int32; q_weight/k_weight [D] or null; cos_sin [max_pos, rot] f32 (cos | sin) or null;
// cache (act dtype) or null; slots [T] int32 (negative = do not write).
// interleaved = 0: the rotation pairs element i with i + rot/2 (neox); 1: element 2i with 2i + 1.
DINFER_API int dinfer_qk_post_styled(void* qkv, int64_t ld, const int* positions, const void* q_weight,
                                     const void* k_weight, float eps, const float* cos_sin, int rot, int interleaved,
                                     void* cache, const int* slots, int block_size,
                                     int T, int H, int Hkv, int D, int act_dtype, int w_dtype,
                                     cudaStream_t stream) {
  if (T < 0 || H <= 0 || Hkv < 0 || D <= 0)
    return refuse(DINFER_BAD_ARGUMENT, "qk_post: bad sizes T=%d H=%d Hkv=%d D=%d", T, H, Hkv, D);
  if (D > MAX_D) return refuse(DINFER_BAD_ARGUMENT, "qk_post: head_dim %d above the limit %d", D, MAX_D);
  if (cos_sin && (rot <= 0 || rot > D || (rot & 1)))
    return refuse(DINFER_BAD_ARGUMENT, "qk_post: rotary dim %d must be even and at most head_dim %d", rot, D);
  if (ld < (int64_t)(H + 2 * Hkv) * D) return refuse(DINFER_BAD_ARGUMENT, "qk_post: row stride below the row's width");
  if (cache && block_size <= 0) return refuse(DINFER_BAD_ARGUMENT, "qk_post: block_size %d", block_size);
  if (T == 0) return 0;
  const int heads = H + 2 * Hkv;
  if ((heads + WARPS - 1) / WARPS > 65535) return refuse(DINFER_BAD_ARGUMENT, "qk_post: too many heads");
  dim3 grid(T, (heads + WARPS - 1) / WARPS);
  DINFER_DISPATCH_DTYPE(act_dtype, TA,
    DINFER_DISPATCH_DTYPE(w_dtype, TW, {
      const bool aligned = ld % 8 == 0 && !(reinterpret_cast<uintptr_t>(qkv) & 31) &&
                           !(reinterpret_cast<uintptr_t>(cache) & 31) && !(reinterpret_cast<uintptr_t>(q_weight) & 31) &&
                           !(reinterpret_cast<uintptr_t>(k_weight) & 31) && !(reinterpret_cast<uintptr_t>(cos_sin) & 31);
      if constexpr (sizeof(TA) == 2) {
        if (aligned && !interleaved && (!cos_sin || rot == D) && D == 128) {
          const int hp = T <= FEW_TOKENS ? 1 : 3;
          const dim3 half_grid(T, (heads + WARPS * 2 * hp - 1) / (WARPS * 2 * hp));
          launch_pdl(hp == 1 ? qk_post_half_warp_kernel<TW, 1> : qk_post_half_warp_kernel<TW, 3>, half_grid, dim3(WARPS * 32), 0,
                     stream, (__nv_bfloat16*)qkv, ld, positions,
                     (const TW*)q_weight, (const TW*)k_weight, eps, cos_sin, (__nv_bfloat16*)cache, slots, block_size, H, Hkv);
          return cuda_status("qk_post");
        }
      }
      if (aligned && !interleaved && (!cos_sin || rot == D) && (D == 32 || D == 64 || D == 128 || D == 256)) {
        const dim3 lanes_grid(T, (heads + WARPS * HPW - 1) / (WARPS * HPW));
        launch_lanes<TA, TW>(lanes_grid, stream, (TA*)qkv, ld, positions, (const TW*)q_weight, (const TW*)k_weight, eps,
                             cos_sin, (TA*)cache, slots, block_size, H, Hkv, D);
        return cuda_status("qk_post");
      }
      // 8-wide accesses need rows, heads and cache slots that start on 32-byte (f32) / 16-byte (bf16) bounds
      const bool vec8 = D % 8 == 0 && ld % 8 == 0 && !(reinterpret_cast<uintptr_t>(qkv) & 31) &&
                        !(reinterpret_cast<uintptr_t>(cache) & 31);
      if (vec8)
        qk_post_kernel<TA, TW, true><<<grid, WARPS * 32, 0, stream>>>(
            (TA*)qkv, ld, positions, (const TW*)q_weight, (const TW*)k_weight, eps, cos_sin, rot, interleaved,
            (TA*)cache, slots, block_size, H, Hkv, D);
      else
        qk_post_kernel<TA, TW, false><<<grid, WARPS * 32, 0, stream>>>(
            (TA*)qkv, ld, positions, (const TW*)q_weight, (const TW*)k_weight, eps, cos_sin, rot, interleaved,
            (TA*)cache, slots, block_size, H, Hkv, D);
      return cuda_status("qk_post");
    }));
  return 0;
}

DINFER_API int dinfer_qk_post(void* qkv, int64_t ld, const int* positions, const void* q_weight,
                              const void* k_weight, float eps, const float* cos_sin, int rot,
                              void* cache, const int* slots, int block_size,
                              int T, int H, int Hkv, int D, int act_dtype, int w_dtype,
                              cudaStream_t stream) {
  return dinfer_qk_post_styled(qkv, ld, positions, q_weight, k_weight, eps, cos_sin, rot, 0, cache, slots, block_size, T, H,
                               Hkv, D, act_dtype, w_dtype, stream);
}

// The general form, for mixers whose keys and values differ in width or whose head norm comes behind the rotation:
// per (token, head) of q (H heads of D), k (Hkv of D) and v (Hkv of Dv), in one pass
//   norm_first:  x <- rms(x) [* w];  x <- rot(x)          (the order of the kernel above)
//   else:        x <- rot(x);        x <- rms(x) [* w]    (norm = 1; the weights may be null: a norm without a weight)
// (x = the projection's output, plus `bias` [(H + Hkv) D + Hkv Dv] f32 where the projection has one);
// q and k written back in place; k and v to the token's slot of a cache [blocks, 2, Hkv, block_size, Dc], whose
// rows are Dc = max(D, Dv) wide (k in the first D, v in the first Dv elements of a row).
// Two more steps, each off unless asked for.  A query temperature: q of a token at position p is multiplied by
// 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1), in 32-bit, last of all.  Mixed values: v <- (1 - lam) v +
// lam v_first with v_first [T, Hkv * Dv] (row stride ld_first) the values another layer made of the same tokens;
// the mixed v is what the cache gets (v in the projection's row is left as it was).  And turned values: with v_cos_sin
// (rows of Dv, like cos_sin) the cached v is rotated over its whole width by its position's row, in the layout of pairs
// of q and k.
namespace {

// x[a], x[b] <- the pair turned by the angle whose cosine and sine are given
__device__ __forceinline__ void turn_pairs(float* xs, const float* cs, int half, int interleaved, int lane) {
  for (int i = lane; i < half; i += 32) {
    const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + half;
    const float c = cs[i], s = cs[half + i];
    const float u = xs[a], v = xs[b];
    xs[a] = u * c - v * s;
    xs[b] = v * c + u * s;
  }
  __syncwarp();
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(WARPS * 32)
qkv_post_general_kernel(TA* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
                        const TW* __restrict__ q_weight, const TW* __restrict__ k_weight, int norm, int norm_first,
                        float eps, const float* __restrict__ cos_sin, int rot, int interleaved, TA* __restrict__ cache,
                        const int* __restrict__ slots, int block_size, int H, int Hkv, int D, int Dv, int Dc,
                        const float* __restrict__ bias, float temp_coef, int temp_every,
                        const TA* __restrict__ v_first, int64_t ld_first, float v_lambda,
                        const float* __restrict__ v_cos_sin) {
  __shared__ float sm[WARPS][MAX_D];
  pdl_enter();
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * WARPS + warp;
  if (head >= H + 2 * Hkv) return;
  const int kind = head < H ? 0 : (head < H + Hkv ? 1 : 2);
  const int width = kind == 2 ? Dv : D;
  const int64_t at = kind == 2 ? (int64_t)(H + Hkv) * D + (int64_t)(head - H - Hkv) * Dv : (int64_t)head * D;
  TA* x = qkv + (int64_t)t * ld + at;
  float* xs = sm[warp];
  // the projection's bias, where it has one, is added here (rounded as the product's own bias kernel would)
  for (int e = lane; e < width; e += 32)
    xs[e] = bias ? to_f32<TA>(from_f32<TA>(to_f32<TA>(x[e]) + bias[at + e])) : to_f32<TA>(x[e]);
  __syncwarp();
  if (kind != 2) {
    const TW* w = kind == 0 ? q_weight : k_weight;
    auto normalize = [&]() {
      float ss = 0.f;
      for (int e = lane; e < D; e += 32) ss += xs[e] * xs[e];
      ss = warp_sum(ss);
      const float rinv = 1.f / sqrtf(ss / (float)D + eps);
      for (int e = lane; e < D; e += 32) xs[e] = xs[e] * rinv * (w ? to_f32<TW>(w[e]) : 1.f);
      __syncwarp();
    };
    if (norm && norm_first) normalize();
    if (cos_sin) turn_pairs(xs, cos_sin + (int64_t)positions[t] * rot, rot >> 1, interleaved, lane);
    if (norm && !norm_first) normalize();
    if (kind == 0 && temp_coef != 0.f) {
      const float f = 1.f + temp_coef * logf((float)((positions[t] + 1) / temp_every) + 1.f);
      for (int e = lane; e < D; e += 32) xs[e] *= f;
    }
    for (int e = lane; e < D; e += 32) x[e] = from_f32<TA>(xs[e]);
  } else if (v_first) {
    const TA* vf = v_first + (int64_t)t * ld_first + (int64_t)(head - H - Hkv) * Dv;
    for (int e = lane; e < Dv; e += 32) xs[e] = (1.f - v_lambda) * xs[e] + v_lambda * to_f32<TA>(vf[e]);
    __syncwarp();
  }
  if (kind == 2 && v_cos_sin) turn_pairs(xs, v_cos_sin + (int64_t)positions[t] * Dv, Dv >> 1, interleaved, lane);
  if (kind != 0 && cache) {
    const int slot = slots[t];
    if (slot < 0) return;
    const int hk = kind == 1 ? head - H : head - H - Hkv;
    const int64_t blk = slot / block_size, off = slot % block_size;
    TA* dst = cache + (((blk * 2 + (kind == 2)) * Hkv + hk) * block_size + off) * Dc;
    for (int e = lane; e < width; e += 32) dst[e] = from_f32<TA>(xs[e]);
  }
}

// The usual case of it in bfloat16 without shared memory: keys and values D = 8 * LPH wide, weighted head norms ahead
// of a rotation in halves, nothing else.  LPH lanes own a head, eight neighbouring elements each (one 16-byte load and
// store); the partner of a rotated element is held by another lane of the head.  (Two or three
// heads a thread, with their loads ahead of the work, measured slower: fewer CTAs fit an SM.)
template <typename TW, int LPH>
__global__ void __launch_bounds__(256)
qkv_post_turn_kernel(__nv_bfloat16* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
                     const TW* __restrict__ q_weight, const TW* __restrict__ k_weight, float eps,
                     const float* __restrict__ cos_sin, int rot, const float* __restrict__ v_cos_sin,
                     __nv_bfloat16* __restrict__ cache, const int* __restrict__ slots, int block_size, int H, int Hkv) {
  constexpr int D = LPH * 8, GROUPS = 256 / LPH;
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int lane = threadIdx.x & 31, l = lane % LPH;
  const int heads = H + 2 * Hkv;
  const int pos = positions[t];
  // this lane's place in a rotation over its head's first n elements: 0 none, 1 the first half, 2 the second
  auto place = [&](int n) { return 8 * l < n / 2 ? 1 : (8 * l < n ? 2 : 0); };
  const int pl_k = cos_sin ? place(rot) : 0, pl_v = v_cos_sin ? place(D) : 0;
  float c_k[8], s_k[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) { c_k[j] = 1.f; s_k[j] = 0.f; }
  if (pl_k) {
    const float* cs = cos_sin + (int64_t)pos * rot + 8 * l - (pl_k == 2 ? rot / 2 : 0);
    load8<float>(cs, c_k);
    load8<float>(cs + rot / 2, s_k);
  }
  const int slot = (cache && slots) ? slots[t] : -1;
  pdl_wait();
  const int head = blockIdx.y * GROUPS + threadIdx.x / LPH;
  const bool live = head < heads;
  const int kind = head < H ? 0 : (head < H + Hkv ? 1 : 2);
  __nv_bfloat16* x = qkv + (int64_t)t * ld + (int64_t)head * D + 8 * l;
  float a[8], c[8], s[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) { a[j] = 0.f; c[j] = c_k[j]; s[j] = s_k[j]; }
  if (live) load8<__nv_bfloat16>(x, a);
  int pl = pl_k, n = rot;
  if (kind == 2) {
    pl = pl_v;
    n = D;
    if (pl) {
      const float* cs = v_cos_sin + (int64_t)pos * D + 8 * l - (pl == 2 ? D / 2 : 0);
      load8<float>(cs, c);
      load8<float>(cs + D / 2, s);
    }
  }
  __syncwarp();
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 8; ++j) ss += a[j] * a[j];
#pragma unroll
  for (int o = LPH / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const TW* w = kind == 0 ? q_weight : k_weight;
  if (live && kind != 2 && w) {
    const float rinv = rsqrtf(ss / (float)D + eps);
    float wv[8];
    load8<TW>(w + 8 * l, wv);
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = a[j] * rinv * wv[j];
  }
  const int other = lane + (pl == 1 ? n / 16 : (pl == 2 ? -(n / 16) : 0));
  float b[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) b[j] = __shfl_sync(0xffffffffu, a[j], other);
  if (pl) {
    const float sign = pl == 1 ? -1.f : 1.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) a[j] = a[j] * c[j] + sign * b[j] * s[j];
  }
  if (live && kind != 2) store8<__nv_bfloat16>(x, a);
  if (live && kind != 0 && slot >= 0) {
    const int hk = kind == 1 ? head - H : head - H - Hkv;
    const int64_t blk = slot / block_size, off = slot % block_size;
    store8<__nv_bfloat16>(cache + (((blk * 2 + (kind == 2)) * Hkv + hk) * block_size + off) * D + 8 * l, a);
  }
}

template <typename TW, int LPH>
void launch_turn(void* qkv, int64_t ld, const int* positions, const void* qw, const void* kw, float eps, const float* cos_sin,
                 int rot, const float* v_cos_sin, void* cache, const int* slots, int block_size, int T, int H, int Hkv,
                 cudaStream_t stream) {
  constexpr int groups = 256 / LPH;
  launch_pdl(qkv_post_turn_kernel<TW, LPH>, dim3(T, (H + 2 * Hkv + groups - 1) / groups), dim3(256), 0, stream, (__nv_bfloat16*)qkv, ld, positions,
             (const TW*)qw, (const TW*)kw, eps, cos_sin, rot, v_cos_sin, (__nv_bfloat16*)cache, slots, block_size, H, Hkv);
}

// ---- what becomes of the heads' outputs: pair m of head h of a token at position p is turned by minus its angle, then
// the head is multiplied by sigmoid(gate[t, h]); 32-bit, one rounding, in place.
template <typename T>
__global__ void __launch_bounds__(256)
heads_out_kernel(T* __restrict__ x, int64_t ldx, const int* __restrict__ positions, const float* __restrict__ cos_sin,
                 const T* __restrict__ gate, int64_t ldg, int H, int Dv, int interleaved) {
  pdl_enter();
  const int t = blockIdx.x;
  const int half = (Dv + 1) / 2;                                  // an odd width has no pairs (and no table)
  const float* cs = cos_sin ? cos_sin + (int64_t)positions[t] * Dv : nullptr;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < H * half; i += gridDim.y * blockDim.x) {
    const int h = i / half, m = i % half;
    const float g = gate ? 1.f / (1.f + expf(-to_f32<T>(gate[(int64_t)t * ldg + h]))) : 1.f;
    T* row = x + (int64_t)t * ldx + (int64_t)h * Dv;
    const int a = interleaved ? 2 * m : m, b = interleaved ? 2 * m + 1 : m + half;
    const float u = to_f32<T>(row[a]), v = b < Dv ? to_f32<T>(row[b]) : 0.f;
    const float c = cs ? cs[m] : 1.f, s = cs ? cs[half + m] : 0.f;
    row[a] = from_f32<T>((u * c + v * s) * g);
    if (b < Dv) row[b] = from_f32<T>((v * c - u * s) * g);
  }
}

// bfloat16, pairs in halves, a width of a multiple of 16: eight pairs a thread, which keeps its cosines and sines while
// it walks over the token's heads
__global__ void __launch_bounds__(256)
heads_out_bf16x8_kernel(__nv_bfloat16* __restrict__ x, int64_t ldx, const int* __restrict__ positions,
                        const float* __restrict__ cos_sin, const __nv_bfloat16* __restrict__ gate, int64_t ldg, int H, int Dv) {
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int half = Dv / 2, per = Dv / 16, groups = 256 / per;
  const int group = threadIdx.x / per, l = threadIdx.x % per;
  float c[8], s[8];
#pragma unroll
  for (int j = 0; j < 8; ++j) { c[j] = 1.f; s[j] = 0.f; }
  if (cos_sin) {
    const float* cs = cos_sin + (int64_t)positions[t] * Dv + 8 * l;
    load8<float>(cs, c);
    load8<float>(cs + half, s);
  }
  pdl_wait();
  if (group >= groups) return;
  for (int h = blockIdx.y * groups + group; h < H; h += gridDim.y * groups) {
    const float g = gate ? 1.f / (1.f + expf(-__bfloat162float(gate[(int64_t)t * ldg + h]))) : 1.f;
    __nv_bfloat16* row = x + (int64_t)t * ldx + (int64_t)h * Dv + 8 * l;
    float u[8], v[8], a[8], b[8];
    load8<__nv_bfloat16>(row, u);
    load8<__nv_bfloat16>(row + half, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) { a[j] = (u[j] * c[j] + v[j] * s[j]) * g; b[j] = (v[j] * c[j] - u[j] * s[j]) * g; }
    store8<__nv_bfloat16>(row, a);
    store8<__nv_bfloat16>(row + half, b);
  }
}

}  // namespace

// x [T, H * Dv] rows of stride ldx (in place); cos_sin f32 [max_pos, Dv] or null; gate [T, H] of x's type, rows of stride
// ldg, or null; positions [T] int32.
DINFER_API int dinfer_heads_out(void* x, int64_t ldx, const int* positions, const float* cos_sin, const void* gate, int64_t ldg,
                                int T, int H, int Dv, int interleaved, int dtype, cudaStream_t stream) {
  if (T < 0 || H <= 0 || Dv <= 0 || ldx < (int64_t)H * Dv || (gate && ldg < H) || (cos_sin && (Dv & 1)))
    return refuse(DINFER_BAD_ARGUMENT, "heads_out: bad sizes T=%d H=%d Dv=%d", T, H, Dv);
  if (T == 0) return 0;
  const auto al = [](const void* q, int n) { return (reinterpret_cast<uintptr_t>(q) & (n - 1)) == 0; };
  if (dtype == DINFER_BF16 && (!interleaved || !cos_sin) && Dv % 16 == 0 && Dv <= 4096 && ldx % 8 == 0 && al(x, 16) && al(cos_sin, 16)) {
    const int groups = 256 / (Dv / 16), all = (H + groups - 1) / groups;
    launch_pdl(heads_out_bf16x8_kernel, dim3(T, T >= 512 ? 1 : all), dim3(256), 0, stream, (__nv_bfloat16*)x, ldx, positions,
               cos_sin, (const __nv_bfloat16*)gate, ldg, H, Dv);
    return cuda_status("heads_out");
  }
  const int64_t pairs = (int64_t)H * ((Dv + 1) / 2);
  const int by = (int)((pairs + 255) / 256 > 64 ? 64 : (pairs + 255) / 256);
  DINFER_DISPATCH_DTYPE(dtype, TA, {
    launch_pdl(heads_out_kernel<TA>, dim3(T, by), dim3(256), 0, stream, (TA*)x, ldx, positions, cos_sin, (const TA*)gate, ldg,
               H, Dv, interleaved);
    return cuda_status("heads_out");
  });
  return 0;
}

DINFER_API int dinfer_qkv_post_turned(void* qkv, int64_t ld, const int* positions, const void* q_weight,
                                     const void* k_weight, int norm, int norm_first, float eps, const float* cos_sin,
                                      int rot, const float* v_cos_sin, int interleaved, void* cache, const int* slots,
                                      int block_size, int T, int H, int Hkv, int D, int Dv, int Dc, const float* bias, float temp_coef,
                                     int temp_every, const void* v_first, int64_t ld_first, float v_lambda,
                                     int act_dtype, int w_dtype, cudaStream_t stream) {
  if (temp_coef != 0.f && temp_every <= 0)
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: the query temperature's step %d must be positive", temp_every);
  if (v_first && ld_first < (int64_t)Hkv * Dv)
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: the first values' row stride is below their width");
  if (T < 0 || H <= 0 || Hkv < 0 || D <= 0 || Dv <= 0 || Dc < D || Dc < Dv)
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: bad sizes T=%d H=%d Hkv=%d D=%d Dv=%d Dc=%d", T, H, Hkv, D, Dv, Dc);
  if (D > MAX_D || Dv > MAX_D) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: head sizes %d / %d above the limit %d", D, Dv, MAX_D);
  if (cos_sin && (rot <= 0 || rot > D || (rot & 1)))
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: rotary dim %d must be even and at most head_dim %d", rot, D);
  if (ld < (int64_t)(H + Hkv) * D + (int64_t)Hkv * Dv) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: row stride below the row's width");
  if (cache && block_size <= 0) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: block_size %d", block_size);
  if (v_cos_sin && (Dv & 1)) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_general: turned values need an even width, got %d", Dv);
  if (T == 0) return 0;
  const auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  // (a rotated half of a multiple of eight elements: the lanes of a pair hold whole runs of it)
  if (act_dtype == DINFER_BF16 && D == Dv && (D == 64 || D == 128 || D == 256) && norm && norm_first && q_weight && k_weight && !interleaved &&
      !bias && temp_coef == 0.f && !v_first && (!cos_sin || rot % 16 == 0) && ld % 8 == 0 && al16(qkv) && al16(cache) &&
      al16(cos_sin) && al16(v_cos_sin) && al16(q_weight) && al16(k_weight)) {
    DINFER_DISPATCH_DTYPE(w_dtype, TW, {
      auto go = D == 64 ? launch_turn<TW, 8> : (D == 128 ? launch_turn<TW, 16> : launch_turn<TW, 32>);
      go(qkv, ld, positions, q_weight, k_weight, eps, cos_sin, rot, v_cos_sin, cache, slots, block_size, T, H, Hkv, stream);
      return cuda_status("qkv_post_turn");
    });
  }
  dim3 grid(T, (H + 2 * Hkv + WARPS - 1) / WARPS);
  DINFER_DISPATCH_DTYPE(act_dtype, TA,
    DINFER_DISPATCH_DTYPE(w_dtype, TW, {
      launch_pdl(qkv_post_general_kernel<TA, TW>, grid, dim3(WARPS * 32), 0, stream, (TA*)qkv, ld, positions,
                 (const TW*)q_weight, (const TW*)k_weight, norm, norm_first, eps, cos_sin, rot, interleaved, (TA*)cache,
                 slots, block_size, H, Hkv, D, Dv, Dc, bias, temp_coef, temp_every, (const TA*)v_first, ld_first, v_lambda,
                 v_cos_sin);
      return cuda_status("qkv_post_general");
    }));
  return 0;
}

DINFER_API int dinfer_qkv_post_general(void* qkv, int64_t ld, const int* positions, const void* q_weight,
                                       const void* k_weight, int norm, int norm_first, float eps, const float* cos_sin,
                                       int rot, int interleaved, void* cache, const int* slots, int block_size, int T,
                                       int H, int Hkv, int D, int Dv, int Dc, const float* bias, int act_dtype,
                                       int w_dtype, cudaStream_t stream) {
  return dinfer_qkv_post_turned(qkv, ld, positions, q_weight, k_weight, norm, norm_first, eps, cos_sin, rot, nullptr, interleaved,
                               cache, slots, block_size, T, H, Hkv, D, Dv, Dc, bias, 0.f, 1, nullptr, 0, 0.f, act_dtype,
                               w_dtype, stream);
}

// One norm over all of q and one over all of k.  Per token: x = the projection's row [q: H * D | k: Hkv * D | v: Hkv * Dv]
// (32-bit or the activations' type), q and k each divided by the root mean square over all their heads at once and
// multiplied by a weight per row of the projection, then rotated by the position's angles; v times v_scale.  q goes to rows
// of its own [T, H * D] in the activations' type, k and v to the token's slot of a cache [blocks, 2, Hkv, block_size, Dc].
// The projection's row is only read, so it may be the 32-bit result of a product that feeds other parts too.
namespace {

constexpr int WHOLE_THREADS = 512;

// V = 4: four neighbouring elements at a time (widths, strides and bases allow it), V = 1: one
template <int V> struct Run { float x[V]; };
template <typename T, int V> __device__ __forceinline__ Run<V> load_run(const T* p) {
  Run<V> r;
  if constexpr (V == 4 && sizeof(T) == 4) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    r.x[0] = a.x; r.x[1] = a.y; r.x[2] = a.z; r.x[3] = a.w;
  } else if constexpr (V == 4) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&a);
    const float2 f0 = __bfloat1622float2(h[0]), f1 = __bfloat1622float2(h[1]);
    r.x[0] = f0.x; r.x[1] = f0.y; r.x[2] = f1.x; r.x[3] = f1.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) r.x[i] = to_f32<T>(p[i]);
  }
  return r;
}
template <typename T, int V> __device__ __forceinline__ void store_run(T* p, const Run<V>& r) {
  if constexpr (V == 4 && sizeof(T) == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(r.x[0], r.x[1], r.x[2], r.x[3]);
  } else if constexpr (V == 4) {
    uint2 a;
    __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&a);
    h[0] = __floats2bfloat162_rn(r.x[0], r.x[1]);
    h[1] = __floats2bfloat162_rn(r.x[2], r.x[3]);
    *reinterpret_cast<uint2*>(p) = a;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = from_f32<T>(r.x[i]);
  }
}

template <typename TI, typename TA, int V>
__global__ void __launch_bounds__(WHOLE_THREADS)
qkv_post_whole_kernel(const TI* __restrict__ qkv, int64_t ld, const int* __restrict__ positions,
                      const float* __restrict__ q_weight, const float* __restrict__ k_weight, float eps,
                      const float* __restrict__ cos_sin, int rot, int interleaved, float v_scale, TA* __restrict__ q_out,
                      TA* __restrict__ cache, const int* __restrict__ slots, int block_size, int H, int Hkv, int D, int Dv,
                      int Dc) {
  __shared__ float red[2][WHOLE_THREADS / 32];
  __shared__ float inv[2];
  pdl_launch_dependents();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int64_t pos = positions[t];
  const int slot = (cache && slots) ? slots[t] : -1;
  pdl_wait();
  const TI* row = qkv + (int64_t)t * ld;
  const int nq = H * D, nk = Hkv * D, nv = Hkv * Dv;
  if (q_weight) {
    float sq = 0.f, sk = 0.f;
    for (int i = tid * V; i < nq + nk; i += WHOLE_THREADS * V) {     // (a run lies in q or in k: both are whole runs)
      const Run<V> a = load_run<TI, V>(row + i);
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < V; ++j) s = fmaf(a.x[j], a.x[j], s);
      if (i < nq) sq += s; else sk += s;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    if (warp < 2) {
      const float v = warp_sum(lane < WHOLE_THREADS / 32 ? red[warp][lane] : 0.f);
      if (lane == 0) inv[warp] = 1.f / sqrtf(v / (float)(warp == 0 ? nq : nk) + eps);
    }
    __syncthreads();
  }
  const int half = cos_sin ? rot >> 1 : 0;
  const float* cs = cos_sin + pos * rot;
  const int64_t blk = slot >= 0 ? slot / block_size : 0, off = slot >= 0 ? slot % block_size : 0;
  // a head's work: its pairs of runs (e, e + half), then the runs that pass unturned
  const int pairs = half / V, units = pairs + (D - 2 * half) / V;
  auto normed = [&](int i) {
    Run<V> a = load_run<TI, V>(row + i);
    if (q_weight) {
      const bool is_q = i < nq;
      const Run<V> w = load_run<float, V>(is_q ? q_weight + i : k_weight + (i - nq));
      const float r = inv[is_q ? 0 : 1];
#pragma unroll
      for (int j = 0; j < V; ++j) a.x[j] = a.x[j] * r * w.x[j];
    }
    return a;
  };
  for (int w = tid; w < (H + Hkv) * units; w += WHOLE_THREADS) {
    const int head = w / units, u = w - head * units;
    TA* dst = nullptr;
    if (head < H) dst = q_out + (int64_t)t * nq + (int64_t)head * D;
    else if (slot >= 0) dst = cache + ((blk * 2 * Hkv + (head - H)) * block_size + off) * Dc;
    if (!dst) continue;
    if (u < pairs) {
      // in halves: elements e.. and e + half..; interleaved (V = 1 only): elements 2 u and 2 u + 1
      const int e0 = interleaved ? 2 * u : u * V, e1 = interleaved ? 2 * u + 1 : u * V + half;
      const Run<V> a = normed(head * D + e0), b = normed(head * D + e1);
      const Run<V> c = load_run<float, V>(cs + u * V), s = load_run<float, V>(cs + half + u * V);
      Run<V> x, y;
#pragma unroll
      for (int j = 0; j < V; ++j) {
        x.x[j] = a.x[j] * c.x[j] - b.x[j] * s.x[j];
        y.x[j] = b.x[j] * c.x[j] + a.x[j] * s.x[j];
      }
      store_run<TA, V>(dst + e0, x);
      store_run<TA, V>(dst + e1, y);
    } else {
      const int e = 2 * half + (u - pairs) * V;
      store_run<TA, V>(dst + e, normed(head * D + e));
    }
  }
  if (slot >= 0)
    for (int i = tid * V; i < nv; i += WHOLE_THREADS * V) {
      Run<V> a = load_run<TI, V>(row + nq + nk + i);
#pragma unroll
      for (int j = 0; j < V; ++j) a.x[j] *= v_scale;
      const int hk = i / Dv;
      store_run<TA, V>(cache + (((blk * 2 + 1) * Hkv + hk) * block_size + off) * Dc + (i - hk * Dv), a);
    }
}

}  // namespace

// qkv [T, >= (H + Hkv) D + Hkv Dv] rows of stride ld in in_dtype; q_weight [H * D] / k_weight [Hkv * D] f32 (both null: no
// norm); cos_sin [positions, rot] f32 or null; q_out [T, H * D] contiguous; cache rows Dc = max(D, Dv) wide.
DINFER_API int dinfer_qkv_post_whole(const void* qkv, int64_t ld, const int* positions, const float* q_weight,
                                     const float* k_weight, float eps, const float* cos_sin, int rot, int interleaved,
                                     float v_scale, void* q_out, void* cache, const int* slots, int block_size, int T, int H,
                                     int Hkv, int D, int Dv, int Dc, int in_dtype, int act_dtype, cudaStream_t stream) {
  if (T < 0 || H <= 0 || Hkv <= 0 || D <= 0 || Dv <= 0 || Dc < D || Dc < Dv || !q_out)
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_whole: bad sizes T=%d H=%d Hkv=%d D=%d Dv=%d Dc=%d", T, H, Hkv, D, Dv, Dc);
  if (cos_sin && (rot <= 0 || rot > D || (rot & 1)))
    return refuse(DINFER_BAD_ARGUMENT, "qkv_post_whole: rotary dim %d must be even and at most head_dim %d", rot, D);
  if (ld < (int64_t)(H + Hkv) * D + (int64_t)Hkv * Dv) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_whole: row stride below the row's width");
  if (cache && (block_size <= 0 || !slots)) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_whole: a cache needs slots and block_size, got %d", block_size);
  if ((q_weight == nullptr) != (k_weight == nullptr)) return refuse(DINFER_BAD_ARGUMENT, "qkv_post_whole: q and k norm weights come together");
  if (T == 0) return 0;
  const auto al16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = D % 8 == 0 && Dv % 4 == 0 && Dc % 4 == 0 && ld % 4 == 0 && (!cos_sin || (rot % 8 == 0 && !interleaved)) &&
                   al16(qkv) && al16(q_out) && al16(cache) && al16(q_weight) && al16(k_weight) && al16(cos_sin);
#define GO(TI, TA, V)                                                                                                      \
  launch_pdl(qkv_post_whole_kernel<TI, TA, V>, dim3(T), dim3(WHOLE_THREADS), 0, stream, (const TI*)qkv, ld, positions,     \
             q_weight, k_weight, eps, cos_sin, rot, interleaved, v_scale, (TA*)q_out, (TA*)cache, slots, block_size, H, Hkv, \
             D, Dv, Dc)
  DINFER_DISPATCH_DTYPE(in_dtype, TI,
    DINFER_DISPATCH_DTYPE(act_dtype, TA, {
      if (vec) GO(TI, TA, 4); else GO(TI, TA, 1);
      return cuda_status("qkv_post_whole");
    }));
#undef GO
  return 0;
}
