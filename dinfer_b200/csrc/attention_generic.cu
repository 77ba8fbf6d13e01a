// Paged causal attention for any head size, any group size, 32-bit or bfloat16 storage:
// the plain-arithmetic path (no tensor cores).  It is the whole attention of the 32-bit model and
// the fallback of the bfloat16 model for head sizes the tensor-core kernels refuse.
//
// One warp owns one (token, query head): the lanes split the head's D elements, keys are visited
// four at a time in position order with an online softmax; scores, softmax and the output sum are
// 32-bit (expf, not the fast intrinsic).  A query at position p sees the keys [max(0, p-window+1), p]
// of its own request (`chunked`: those of its own chunk of `window` positions), read through the request's block table.  Values may be Dv wide where keys are D wide (the
// cache's rows are then Dc = max(D, Dv) wide); with `sink` the softmax has one more term of score 0 and no value:
// p_j = exp(s_j) / (1 + sum exp(s_j)); `sinks` gives that term a score of its own per query head.  With `slopes` (one number per query head) a distance bias is taken off every
// score: s_ij - slopes[h] * (i - j).  `keep`: behind a window the keys below it are seen too.  `softcap` > 0: a score is
// softcap * tanh(score / softcap), ahead of the bias.
//
// Counterpart in the reference: the any-D reference kernels crates/kernels/cuda/gqa.cu:956-1118.
#include "common.cuh"

using namespace dinfer;

namespace {

constexpr int WARPS = 4;
constexpr int KEYS = 4;

template <typename T, int C>   // C = ceil(max(D, Dv) / 32) elements per lane
__global__ void __launch_bounds__(WARPS * 32)
attention_generic_kernel(const T* __restrict__ q, int64_t ldq, T* __restrict__ out, int64_t ldo,
                         const T* __restrict__ cache, const int* __restrict__ block_table, int max_blocks,
                         const int* __restrict__ cu_seqlens, const int* __restrict__ positions,
                         int num_reqs, int H, int Hkv, int D, int Dv, int Dc, int block_size, float scale, int window,
                         int chunked, int keep, float softcap, int sink, const float* __restrict__ sinks,
                         const float* __restrict__ slopes) {
  const int t = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y * WARPS + warp;
  if (h >= H) return;
  // request of this token: last b with cu_seqlens[b] <= t
  int lo = 0, hi = num_reqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_seqlens[mid] <= t) lo = mid; else hi = mid - 1;
  }
  const int* table = block_table + (int64_t)lo * max_blocks;
  const int hk = h / (H / Hkv);
  const int pos = positions[t];
  const int first = first_key(pos, window, chunked);
  const float slope = slopes ? slopes[h] : 0.f;

  float qv[C], acc[C];
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int e = lane + 32 * c;
    qv[c] = e < D ? to_f32<T>(q[(int64_t)t * ldq + (int64_t)h * D + e]) * scale : 0.f;
    acc[c] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int64_t plane = (int64_t)Hkv * block_size * Dc;      // one of k / v of one block
  const int kept = min(keep, first);                           // the kept keys in front of the window, then the window
  const int visits = kept + pos - first + 1;
  for (int n0 = 0; n0 < visits; n0 += KEYS) {
    const T* kp[KEYS];
    float s[KEYS];
#pragma unroll
    for (int u = 0; u < KEYS; ++u) {
      const int j = n0 + u < kept ? n0 + u : first + n0 + u - kept;
      kp[u] = nullptr;
      s[u] = 0.f;
      // a page the table does not hold (-1: a dummy row of a captured graph, a page a window has passed) is no key
      const int64_t blk = j <= pos ? table[j / block_size] : -1;
      if (blk >= 0) {
        kp[u] = cache + blk * 2 * plane + ((int64_t)hk * block_size + j % block_size) * Dc;
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const int e = lane + 32 * c;
          if (e < D) s[u] += qv[c] * to_f32<T>(kp[u][e]);
        }
      }
    }
#pragma unroll
    for (int u = 0; u < KEYS; ++u) {
      const int j = n0 + u < kept ? n0 + u : first + n0 + u - kept;
      if (!kp[u]) { s[u] = -INFINITY; continue; }
      s[u] = warp_sum(s[u]);
      if (softcap > 0.f) s[u] = softcap * tanhf(s[u] / softcap);
      s[u] -= slope * (float)(pos - j);
    }
    float m_new = m;
#pragma unroll
    for (int u = 0; u < KEYS; ++u) m_new = fmaxf(m_new, s[u]);
    if (m_new == -INFINITY) continue;                            // no key so far
    const float alpha = expf(m - m_new);
    l *= alpha;
#pragma unroll
    for (int c = 0; c < C; ++c) acc[c] *= alpha;
#pragma unroll
    for (int u = 0; u < KEYS; ++u) {
      if (kp[u]) {
        const float p = expf(s[u] - m_new);
        l += p;
        const T* vp = kp[u] + plane;
#pragma unroll
        for (int c = 0; c < C; ++c) {
          const int e = lane + 32 * c;
          if (e < Dv) acc[c] += p * to_f32<T>(vp[e]);
        }
      }
    }
    m = m_new;
  }
  if (sink) {                                                     // one more term, exp(score - m), in the denominator only
    const float extra = sinks ? sinks[h] : 0.f;
    const float m_new = fmaxf(m, extra);
    const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
    l = l * alpha + expf(extra - m_new);
#pragma unroll
    for (int c = 0; c < C; ++c) acc[c] *= alpha;
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;                      // a row without keys gives zeros
#pragma unroll
  for (int c = 0; c < C; ++c) {
    const int e = lane + 32 * c;
    if (e < Dv) out[(int64_t)t * ldo + (int64_t)h * Dv + e] = from_f32<T>(acc[c] * inv);
  }
}

template <typename T, int C>
int launch(const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache, const int* block_table,
           int max_blocks, const int* cu_seqlens, const int* positions, int T_, int B, int H, int Hkv,
           int D, int Dv, int Dc, int block_size, float scale, int window, int chunked, int keep, float softcap, int sink,
           const float* sinks, const float* slopes, cudaStream_t stream) {
  dim3 grid(T_, (H + WARPS - 1) / WARPS);
  attention_generic_kernel<T, C><<<grid, WARPS * 32, 0, stream>>>(
      (const T*)q, ldq, (T*)out, ldo, (const T*)cache, block_table, max_blocks, cu_seqlens, positions,
      B, H, Hkv, D, Dv, Dc, block_size, scale, window, chunked, keep, softcap, sink, sinks, slopes);
  return cuda_status("attention_generic");
}

}  // namespace

DINFER_DEFINE_LAST_ERROR()

DINFER_API int dinfer_attention_generic_bias(const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache,
                                             const int* block_table, int max_blocks, const int* cu_seqlens,
                                             const int* positions, int T, int B, int H, int Hkv, int D, int Dv, int Dc,
                                             int block_size, float scale, int window, int chunked, int keep_first, float softcap,
                                             int sink, const float* sinks, const float* slopes, int dtype, cudaStream_t stream);

// q: [T, ...] rows of stride ldq, head h at h*D; out likewise with stride ldo.
// cache [num_blocks, 2, Hkv, block_size, D]; block_table [B, max_blocks] int32;
// cu_seqlens [B+1] int32 (token offsets of the requests); positions [T] int32.
// window <= 0: all keys.
DINFER_API int dinfer_attention_generic(const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache,
                                        const int* block_table, int max_blocks, const int* cu_seqlens,
                                        const int* positions, int T, int B, int H, int Hkv, int D,
                                        int block_size, float scale, int window, int dtype,
                                        cudaStream_t stream) {
  return dinfer_attention_generic_bias(q, ldq, out, ldo, cache, block_table, max_blocks, cu_seqlens, positions, T, B, H,
                                       Hkv, D, D, D, block_size, scale, window, 0, 0, 0.f, 0, nullptr, nullptr, dtype, stream);
}

// The same with values Dv wide in a cache whose rows are Dc wide (out: head h at h*Dv), and an optional sink.
DINFER_API int dinfer_attention_generic_ex(const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache,
                                           const int* block_table, int max_blocks, const int* cu_seqlens,
                                           const int* positions, int T, int B, int H, int Hkv, int D, int Dv, int Dc,
                                           int block_size, float scale, int window, int sink, int dtype,
                                           cudaStream_t stream) {
  return dinfer_attention_generic_bias(q, ldq, out, ldo, cache, block_table, max_blocks, cu_seqlens, positions, T, B, H,
                                       Hkv, D, Dv, Dc, block_size, scale, window, 0, 0, 0.f, sink, nullptr, nullptr, dtype, stream);
}

// The same with a distance bias (slopes [H] f32 or null), keys by chunks (chunked, see first_key), kept first keys
// (keep_first > 0, with a window), a soft cap on the scores (softcap > 0) and a score per head
// for the sink's term (sinks [H] f32 or null: 0).
DINFER_API int dinfer_attention_generic_bias(const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache,
                                             const int* block_table, int max_blocks, const int* cu_seqlens,
                                             const int* positions, int T, int B, int H, int Hkv, int D, int Dv, int Dc,
                                             int block_size, float scale, int window, int chunked, int keep_first, float softcap,
                                             int sink, const float* sinks, const float* slopes, int dtype, cudaStream_t stream) {
  if (keep_first < 0 || !(softcap >= 0.f) || (keep_first > 0 && chunked))
    return refuse(DINFER_BAD_ARGUMENT, "attention_generic: keep_first %d, softcap %g (kept keys belong to a window)", keep_first, (double)softcap);
  const int keep = window > 0 ? keep_first : 0;
  if (Dv <= 0 || Dc < D || Dc < Dv) return refuse(DINFER_BAD_ARGUMENT, "attention_generic: bad sizes D=%d Dv=%d Dc=%d", D, Dv, Dc);
  if (T < 0 || B <= 0 || H <= 0 || Hkv <= 0 || D <= 0 || block_size <= 0 || max_blocks <= 0)
    return refuse(DINFER_BAD_ARGUMENT, "attention_generic: bad sizes T=%d B=%d H=%d Hkv=%d D=%d block=%d",
                  T, B, H, Hkv, D, block_size);
  if (H % Hkv) return refuse(DINFER_BAD_ARGUMENT, "attention_generic: heads %d not divisible by kv heads %d", H, Hkv);
  if (D > 512 || Dv > 512) return refuse(DINFER_BAD_ARGUMENT, "attention_generic: head_dim %d / %d above the limit 512", D, Dv);
  if ((H + WARPS - 1) / WARPS > 65535) return refuse(DINFER_BAD_ARGUMENT, "attention_generic: too many heads");
  if (T == 0) return 0;
  const int c = ((D > Dv ? D : Dv) + 31) / 32;
#define GO(C) return launch<T_, C>(q, ldq, out, ldo, cache, block_table, max_blocks, cu_seqlens, positions, \
                                   T, B, H, Hkv, D, Dv, Dc, block_size, scale, window, chunked, keep, softcap, sink, sinks, slopes, stream)
  DINFER_DISPATCH_DTYPE(dtype, T_, {
    if (c <= 1) GO(1);
    else if (c <= 2) GO(2);
    else if (c <= 4) GO(4);
    else if (c <= 8) GO(8);
    else GO(16);
  });
#undef GO
  return 0;
}
