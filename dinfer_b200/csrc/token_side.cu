// Around a layer's token input, a small vector per token and layer that joins the stream behind the layer's sublayers
// (x <- x + norm(W_proj (gelu_tanh(W_gate x) * e)), e = the layer's part of the token's row of a table):
//
//   branch_join   x += a (+ f), the branches of a layer whose sublayers read one norm, in 32-bit; the sum also rounded to
//                 the activation type, for the product that reads the stream itself
//   token_gate    out[t, j] = gelu_tanh(g[t, j]) * table[id_t, at + j]; the table row of the step's token ids, an id
//                 -(r + 1) standing for prev[r] (a token the previous step sampled, still on the device)
//
// The norm, the add and the next layer's norm behind them are the join kernel of the sandwich arrangement.
#include "common.cuh"

using namespace dinfer;

namespace {

template <typename TA>
__global__ void __launch_bounds__(256)
branch_join_kernel(float* __restrict__ x, const TA* __restrict__ a, const TA* __restrict__ f, TA* __restrict__ cast, int64_t n) {
  pdl_enter();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    float v = x[i] + to_f32<TA>(a[i]);
    if (f) v += to_f32<TA>(f[i]);
    x[i] = v;
    if (cast) cast[i] = from_f32<TA>(v);
  }
}

// bfloat16 branches, eight elements (16 bytes of a branch, 32 of the stream) a thread
__global__ void __launch_bounds__(256)
branch_join_bf16x8_kernel(float4* __restrict__ x, const uint4* __restrict__ a, const uint4* __restrict__ f, uint4* __restrict__ cast,
                          int64_t n8) {
  pdl_enter();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n8; i += (int64_t)gridDim.x * blockDim.x) {
    const float4 x0 = x[2 * i], x1 = x[2 * i + 1];
    float v[8] = {x0.x, x0.y, x0.z, x0.w, x1.x, x1.y, x1.z, x1.w};
    auto add = [&](const uint4& u) {
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
      for (int j = 0; j < 4; ++j) { const float2 y = __bfloat1622float2(p[j]); v[2 * j] += y.x; v[2 * j + 1] += y.y; }
    };
    const uint4 av = a[i];
    uint4 fv = make_uint4(0, 0, 0, 0);
    if (f) fv = f[i];
    add(av);
    if (f) add(fv);
    x[2 * i] = make_float4(v[0], v[1], v[2], v[3]);
    x[2 * i + 1] = make_float4(v[4], v[5], v[6], v[7]);
    if (cast) {
      uint4 o;
      __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
      for (int j = 0; j < 4; ++j) p[j] = __floats2bfloat162_rn(v[2 * j], v[2 * j + 1]);
      cast[i] = o;
    }
  }
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(256)
token_gate_kernel(const TA* __restrict__ g, int64_t ldg, const int* __restrict__ ids, const int* __restrict__ prev, int prev_rows,
                  const TW* __restrict__ table, int64_t ld_table, int vocab, int at, TA* __restrict__ out, int T, int dim) {
  pdl_enter();
  const int64_t n = (int64_t)T * dim;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / dim;
    const int j = (int)(i - t * dim);
    int id = ids[t];
    if (id < 0 && prev && -id - 1 < prev_rows) id = prev[-id - 1];
    if (id < 0 || id >= vocab) id = 0;
    const float z = to_f32<TA>(g[t * ldg + j]);
    const float gate = 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
    out[i] = from_f32<TA>(gate * to_f32<TW>(table[(int64_t)id * ld_table + at + j]));
  }
}

}  // namespace

DINFER_DEFINE_LAST_ERROR()

// x f32 [n] += a [n] (+ f [n] or null), in place; cast [n] of the branches' type or null gets the sums rounded.
DINFER_API int dinfer_branch_join(float* x, const void* a, const void* f, void* cast, int64_t n, int act_dtype, cudaStream_t stream) {
  if (n < 0 || !x || !a) return refuse(DINFER_BAD_ARGUMENT, "branch_join: bad arguments n=%lld", (long long)n);
  if (n == 0) return 0;
  const auto al = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = act_dtype == DINFER_BF16 && n % 8 == 0 && al(x) && al(a) && al(f) && al(cast);
  const int64_t items = vec ? n / 8 : n;
  const int blocks = (int)((items + 255) / 256 < 16384 ? (items + 255) / 256 : 16384);
  if (vec) {
    launch_pdl(branch_join_bf16x8_kernel, dim3(blocks), dim3(256), 0, stream, (float4*)x, (const uint4*)a, (const uint4*)f,
               (uint4*)cast, items);
    return cuda_status("branch_join");
  }
  DINFER_DISPATCH_DTYPE(act_dtype, TA, {
    launch_pdl(branch_join_kernel<TA>, dim3(blocks), dim3(256), 0, stream, x, (const TA*)a, (const TA*)f, (TA*)cast, n);
    return cuda_status("branch_join");
  });
  return 0;
}

// g [T, dim] rows of stride ldg; ids [T]; prev [prev_rows] or null; table [vocab, >= at + dim] rows of stride ld_table; out
// [T, dim] contiguous.
DINFER_API int dinfer_token_gate(const void* g, int64_t ldg, const int* ids, const int* prev, int prev_rows, const void* table,
                                 int64_t ld_table, int vocab, int at, void* out, int T, int dim, int act_dtype, int w_dtype,
                                 cudaStream_t stream) {
  if (T < 0 || dim <= 0 || vocab <= 0 || at < 0 || ldg < dim || ld_table < (int64_t)at + dim)
    return refuse(DINFER_BAD_ARGUMENT, "token_gate: bad sizes T=%d dim=%d at=%d vocab=%d", T, dim, at, vocab);
  if (T == 0) return 0;
  const int64_t n = (int64_t)T * dim;
  const int blocks = (int)((n + 255) / 256 < 8192 ? (n + 255) / 256 : 8192);
  DINFER_DISPATCH_DTYPE(act_dtype, TA,
    DINFER_DISPATCH_DTYPE(w_dtype, TW, {
      launch_pdl(token_gate_kernel<TA, TW>, dim3(blocks), dim3(256), 0, stream, (const TA*)g, ldg, ids, prev, prev_rows,
                 (const TW*)table, ld_table, vocab, at, (TA*)out, T, dim);
      return cuda_status("token_gate");
    }));
  return 0;
}
