// A state-space mixer with one decay per head and token (Mamba-2's form): per head a matrix S [N, P] in 32-bit is carried
// from token to token of a request, beside the last (taps - 1) inputs of a short causal convolution.  A token's projected
// row is [z: inner | x: inner | B: G * N | C: G * N | dt: H] with inner = H * P; x, B and C pass the convolution (with a
// bias) and silu; head h uses B and C of group h / (H / G):
//
//     dt = softplus(dt + dt_bias_h),   S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T,   y_t = S_t^T C_t + D_h x_t
//
// and what leaves the mixer ahead of its output projection is y * silu(z), RMS-normed in `parts` equal parts of the row.
//
//   ssm_step      requests that bring one token: convolution, step size, state and read-out in one launch, a CTA per
//                 (request, head, run of columns).  S goes through registers: its loads are asked for before the kernels
//                 in front have finished (no kernel of a step but this one touches a single token's S, and none in
//                 front of it its convolution's inputs), each element is read and written once.  The decay is applied as S + S * expm1(..), which keeps the digits of a decay just below one.
//   ssm_prep      requests that bring more: convolution and silu of x, B, C; dt and the decay's logarithm
//   ssm_sums, ssm_scan, ssm_outputs
//                 their chunks of 64 tokens side by side.  With c_t the running sum of the decays' logarithms inside a
//                 chunk, n its tokens and S the state before it:
//                     U    = sum_s exp(c_n - c_s) dt_s B_s x_s^T              per (chunk, head): needs no state
//                     S   <- exp(c_n) S + U                                   a walk over the chunks per element of S
//                     y_t  = sum_(s<=t) (C_t . B_s) exp(c_t - c_s) dt_s x_s + exp(c_t) S^T C_t + D x_t
//                 C_t . B_s is the same for all heads of a group: ssm_sums makes it once per (chunk, group).  The running
//                 sums are 64-bit, so that a difference of two large ones is exact where strong and weak decays follow
//                 one another; everything else is 32-bit.
//   ssm_post      gate and norm; and each request's last convolution inputs move into its state.
//
// A request whose `fresh` flag is set starts from zeros whatever its slot holds.  What a token gets depends on how a
// request is cut into steps through the order of sums only.
#include "common.cuh"

using namespace dinfer;

namespace {

constexpr int THREADS = 256;
constexpr int CP = 64;           // tokens per chunk
constexpr int TP = 64;           // tile edge: state channels x value columns (sums), tokens x value columns (outputs)
constexpr int KT = 32;           // state channels per pass of the outputs kernel
constexpr int LDT = TP + 4;      // row stride of the transposed tiles (rows stay 16-byte aligned)

struct Params {
  const float* P; int64_t ldp;                     // projected rows
  const float* conv_w; const float* conv_b;        // [channels, taps], [channels]; channels = inner + 2 G N
  const float* dt_bias; const float* A_log; const float* D;   // [H]
  float* state; int64_t ld_state; int hist;        // rows: S [H, N, P], then from `hist` on the convolution's inputs
  const int* cu; const int* slots; const int* fresh;
  float* y;                                        // [T, inner]
  float* xbc; float* dt; float* la;                // [T, channels], [T, H], [T, H] (ssm_prep)
  float* U; float* cb; float* decay;               // work of the chunks: [slot][H][N][P], [slot][G][CP][CP], [slot][H]
  int T, B, H, G, N, Pd, taps;
  __host__ __device__ int inner() const { return H * Pd; }
  __host__ __device__ int channels() const { return H * Pd + 2 * G * N; }
};

__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.f ? z : log1pf(expf(z)); }

template <int V> struct alignas(4 * V) Vec { float x[V]; };
template <int V> __device__ __forceinline__ Vec<V> ldv(const float* p) { return *reinterpret_cast<const Vec<V>*>(p); }
template <int V> __device__ __forceinline__ void stv(float* p, const Vec<V>& v) { *reinterpret_cast<Vec<V>*>(p) = v; }

// ---------------------------------------------------------------- one token
// L lanes share a row of S, V neighbouring columns each; 256 / L rows at a time.  RPT > 0: a thread's rows (at most RPT)
// stay in registers from the loads ahead of the wait on; RPT = 0: rows as they come.
template <int V, int L, int RPT>
__global__ void __launch_bounds__(THREADS, RPT == 16 ? 2 : (RPT == 8 ? 3 : 4)) ssm_step_kernel(const Params p) {
  constexpr int PT = V * L, R = THREADS / L, WARPS = THREADS / 32;
  extern __shared__ float sm[];                    // B [N], C [N], x [PT], partial sums [WARPS][PT]
  float* sB = sm;
  float* sC = sB + p.N;
  float* sx = sC + p.N;
  float* red = sx + PT;
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * PT;
  const int t = p.cu[b];
  if (p.cu[b + 1] - t != 1) return;                // portions are the chunk kernels'
  const int tid = threadIdx.x, col = (tid % L) * V, r0 = tid / L;
  const bool is_fresh = p.fresh[b] != 0;
  float* row_state = p.state + (int64_t)p.slots[b] * p.ld_state;
  float* S = row_state + (int64_t)h * p.N * p.Pd + c0 + col;
  const bool live = c0 + col < p.Pd;               // (V divides P)
  Vec<V> s[RPT > 0 ? RPT : 1];
  if constexpr (RPT > 0) {
#pragma unroll
    for (int k = 0; k < RPT; ++k) {
      const int r = r0 + k * R;
#pragma unroll
      for (int e = 0; e < V; ++e) s[k].x[e] = 0.f;
      if (live && r < p.N && !is_fresh) s[k] = ldv<V>(S + (int64_t)r * p.Pd);
    }
  }
  const float* hist = row_state + p.hist;
  const int inner = p.inner(), ch = p.channels(), g = h / (p.H / p.G);
  auto channel = [&](int i) {                                       // of x | B | C; -1: none
    if (i < p.N) return inner + g * p.N + i;
    if (i < 2 * p.N) return inner + (p.G + g) * p.N + i - p.N;
    return c0 + i - 2 * p.N < p.Pd ? h * p.Pd + c0 + i - 2 * p.N : -1;
  };
  // the convolution's part of earlier inputs, which no kernel in front of this one writes either; each thread ends what it began
  for (int i = tid; i < 2 * p.N + PT; i += THREADS) {
    const int c = channel(i);
    float a = 0.f;
    if (c >= 0) {
      const float* w = p.conv_w + (int64_t)c * p.taps;
      a = p.conv_b[c];
      if (!is_fresh)
        for (int d = 0; d < p.taps - 1; ++d) a = fmaf(w[d], hist[(int64_t)d * ch + c], a);
    }
    sm[i] = a;
  }
  pdl_wait();
  const float* row = p.P + (int64_t)t * p.ldp + inner;             // the convolution's inputs
  for (int i = tid; i < 2 * p.N + PT; i += THREADS) {
    const int c = channel(i);
    if (c >= 0) sm[i] = silu_f(fmaf(p.conv_w[(int64_t)c * p.taps + p.taps - 1], row[c], sm[i]));
  }
  const float dt = softplus_f(row[ch + h] + p.dt_bias[h]);
  const float g1 = expm1f(-expf(p.A_log[h]) * dt);
  __syncthreads();
  Vec<V> x, acc;
#pragma unroll
  for (int e = 0; e < V; ++e) { x.x[e] = sx[col + e]; acc.x[e] = 0.f; }
  auto update = [&](int r, Vec<V>& v) {
    const float kb = dt * sB[r], c = sC[r];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      v.x[e] = fmaf(kb, x.x[e], fmaf(v.x[e], g1, v.x[e]));
      acc.x[e] = fmaf(v.x[e], c, acc.x[e]);
    }
    stv<V>(S + (int64_t)r * p.Pd, v);
  };
  if (live) {
    if constexpr (RPT > 0) {
#pragma unroll
      for (int k = 0; k < RPT; ++k)
        if (r0 + k * R < p.N) update(r0 + k * R, s[k]);
    } else {
#pragma unroll 4
      for (int r = r0; r < p.N; r += R) {
        Vec<V> v;
#pragma unroll
        for (int e = 0; e < V; ++e) v.x[e] = 0.f;
        if (!is_fresh) v = ldv<V>(S + (int64_t)r * p.Pd);
        update(r, v);
      }
    }
  }
#pragma unroll
  for (int o = L; o < 32; o <<= 1)
#pragma unroll
    for (int e = 0; e < V; ++e) acc.x[e] += __shfl_xor_sync(0xffffffffu, acc.x[e], o);
  if ((tid & 31) < L)
#pragma unroll
    for (int e = 0; e < V; ++e) red[(tid >> 5) * PT + col + e] = acc.x[e];
  __syncthreads();
  if (tid < PT && c0 + tid < p.Pd) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) o += red[w * PT + tid];
    p.y[(int64_t)t * inner + (int64_t)h * p.Pd + c0 + tid] = fmaf(p.D[h], sx[tid], o);
  }
}

// ---------------------------------------------------------------- portions: inputs
__device__ __forceinline__ int request_of(const int* __restrict__ cu, int B, int t) {
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

constexpr int PREP_THREADS = 128, PREP_TOKENS = 16;

// grid (runs of 16 tokens, runs of channels + 1); the last blockIdx.y makes dt and the decay's logarithm.  A thread walks
// its V channels over the run's tokens with the TAPS - 1 inputs before them in registers (TAPS = 0: any number of taps).
template <int V, int TAPS>
__global__ void __launch_bounds__(PREP_THREADS) ssm_prep_kernel(const Params p) {
  pdl_enter();
  const int t0 = blockIdx.x * PREP_TOKENS, t1 = min(p.T, t0 + PREP_TOKENS);
  const int inner = p.inner(), ch = p.channels();
  int b = request_of(p.cu, p.B, t0);
  if (blockIdx.y == gridDim.y - 1) {
    for (int i = threadIdx.x; i < (t1 - t0) * p.H; i += PREP_THREADS) {
      const int t = t0 + i / p.H, h = i % p.H;
      const float dt = softplus_f(p.P[(int64_t)t * p.ldp + inner + ch + h] + p.dt_bias[h]);
      p.dt[(int64_t)t * p.H + h] = dt;
      p.la[(int64_t)t * p.H + h] = -expf(p.A_log[h]) * dt;
    }
    return;
  }
  const int c = (blockIdx.y * PREP_THREADS + threadIdx.x) * V;
  if (c >= ch) return;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  constexpr int KEEP = TAPS > 1 ? TAPS - 1 : 1;
  float w[V][TAPS > 0 ? TAPS : 1], bias[V];
  Vec<V> before[KEEP];                              // before[d]: the input d + 1 tokens back
#pragma unroll
  for (int e = 0; e < V; ++e) {
    bias[e] = p.conv_b[c + e];
    if constexpr (TAPS > 0)
#pragma unroll
      for (int d = 0; d < TAPS; ++d) w[e][d] = p.conv_w[(int64_t)(c + e) * TAPS + d];
  }
  int start = p.cu[b], end = p.cu[b + 1];
  bool load = true;                                 // the inputs before the next token are not in registers
  for (int t = t0; t < t1; ++t) {
    while (t >= end && b + 1 < p.B) { ++b; start = end; end = p.cu[b + 1]; load = true; }
    if (end - start == 1 || t >= end) continue;     // single tokens are ssm_step's
    const float* x = p.P + (int64_t)t * p.ldp + inner + c;
    const float* hist = p.state + (int64_t)p.slots[b] * p.ld_state + p.hist;
    const bool have = !p.fresh[b];
    auto input = [&](int d) {                       // d tokens back: from the step, or from the request's state
      Vec<V> v;
#pragma unroll
      for (int e = 0; e < V; ++e) v.x[e] = 0.f;
      const int i = t - start - d;
      if (i >= 0) v = ldv<V>(x - (int64_t)d * p.ldp);
      else if (have) {
#pragma unroll
        for (int e = 0; e < V; ++e) v.x[e] = hist[(int64_t)(taps - 1 + i) * ch + c + e];
      }
      return v;
    };
    const Vec<V> now = ldv<V>(x);
    Vec<V> o;
#pragma unroll
    for (int e = 0; e < V; ++e) o.x[e] = bias[e];
    if constexpr (TAPS > 0) {
      if (load) {
#pragma unroll
        for (int d = 1; d < TAPS; ++d) before[d - 1] = input(d);
        load = false;
      }
#pragma unroll
      for (int d = TAPS - 1; d > 0; --d)
#pragma unroll
        for (int e = 0; e < V; ++e) o.x[e] = fmaf(w[e][TAPS - 1 - d], before[d - 1].x[e], o.x[e]);
#pragma unroll
      for (int e = 0; e < V; ++e) o.x[e] = silu_f(fmaf(w[e][TAPS - 1], now.x[e], o.x[e]));
#pragma unroll
      for (int d = TAPS - 1; d > 1; --d) before[d - 1] = before[d - 2];
      if constexpr (TAPS > 1) before[0] = now;
    } else {
      for (int d = taps - 1; d > 0; --d) {
        const Vec<V> v = input(d);
#pragma unroll
        for (int e = 0; e < V; ++e) o.x[e] = fmaf(p.conv_w[(int64_t)(c + e) * taps + taps - 1 - d], v.x[e], o.x[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) o.x[e] = silu_f(fmaf(p.conv_w[(int64_t)(c + e) * taps + taps - 1], now.x[e], o.x[e]));
    }
    stv<V>(p.xbc + (int64_t)t * ch + c, o);
  }
}

// ---------------------------------------------------------------- portions: chunks side by side
// request b's chunk c lives in work slot t_begin / CP + b + c: slots of different requests never meet, and there are at
// most T / CP + B of them
__device__ __forceinline__ int64_t chunk_slot(int t_begin, int b, int c) { return (int64_t)(t_begin / CP + b + c); }

// c_t of a chunk (64-bit) by one warp: two tokens a lane
__device__ __forceinline__ void chunk_log_decay(const float* la, int64_t ld, int n, double* cum) {
  const int lane = threadIdx.x & 31;
  const double a0 = 2 * lane < n ? (double)la[(int64_t)(2 * lane) * ld] : 0.0;
  const double a1 = 2 * lane + 1 < n ? (double)la[(int64_t)(2 * lane + 1) * ld] : 0.0;
  double s = a0 + a1;
#pragma unroll
  for (int d = 1; d < 32; d <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, s, d);
    if (lane >= d) s += v;
  }
  cum[2 * lane] = s - a1;
  cum[2 * lane + 1] = s;
}

// four neighbouring elements of which `left` are there (the others read as zeros); VEC: all four or none, 16-byte aligned
template <bool VEC>
__device__ __forceinline__ float4 load4(const float* p, int left) {
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  if (VEC) {
    if (left > 0) v = *reinterpret_cast<const float4*>(p);
  } else {
    if (left > 0) v.x = p[0];
    if (left > 1) v.y = p[1];
    if (left > 2) v.z = p[2];
    if (left > 3) v.w = p[3];
  }
  return v;
}
template <bool VEC>
__device__ __forceinline__ void store4(float* p, int left, const float (&v)[4]) {
  if (VEC) {
    if (left > 0) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (left > u) p[u] = v[u];
  }
}
__device__ __forceinline__ float4 get4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void put4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }

// grid (chunks, H * tiles + G, B): a 64 x 64 tile of U for one (chunk, head), or the scores C_t . B_s of one (chunk, group)
template <bool VEC>
__global__ void __launch_bounds__(THREADS) ssm_sums_kernel(const Params p) {
  __shared__ __align__(16) float a_s[CP][LDT];     // [token][state channel] of B
  __shared__ __align__(16) float b_s[CP][LDT];     // [token][value column], scaled; or [token][state channel] of C
  __shared__ double cum[CP];
  __shared__ float wgt[CP];
  pdl_enter();
  const int tiles_n = (p.N + TP - 1) / TP, tiles_v = (p.Pd + TP - 1) / TP;
  const int b = blockIdx.z, c = blockIdx.x, tid = threadIdx.x;
  const int t_begin = p.cu[b], t_end = p.cu[b + 1];
  const int t0 = t_begin + c * CP;
  if (t_end - t_begin <= 1 || t0 >= t_end) return;
  const int n = min(CP, t_end - t0), ch = p.channels(), inner = p.inner();
  const int64_t slot = chunk_slot(t_begin, b, c);
  const int ty = tid >> 4, tx = tid & 15;
  const int ls = tid >> 4, le = (tid & 15) * 4;    // this thread's place in a tile it loads: rows ls + 16 k, columns le ..
  float acc[4][4] = {};
  const int job = (int)blockIdx.y - p.H * tiles_n * tiles_v;
  if (job >= 0) {
    // ---- scores of group `job`: rows t = 4 ty + i, columns s = tx + 16 j (neighbouring lanes read neighbouring rows)
    const float* Bp = p.xbc + (int64_t)t0 * ch + inner + job * p.N;
    const float* Cp = Bp + p.G * p.N;
    for (int e0 = 0; e0 < p.N; e0 += CP) {
      __syncthreads();
#pragma unroll
      for (int k = 0; k < CP / 16; ++k) {
        const int s = ls + 16 * k, left = s < n ? p.N - e0 - le : 0;
        put4(&a_s[s][le], load4<VEC>(Bp + (int64_t)s * ch + e0 + le, left));
        put4(&b_s[s][le], load4<VEC>(Cp + (int64_t)s * ch + e0 + le, left));
      }
      __syncthreads();
      const int ne = min(CP, p.N - e0);
      for (int e = 0; e < ne; e += 4) {
        float4 q[4], k4[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) { q[i] = get4(&b_s[ty * 4 + i][e]); k4[i] = get4(&a_s[tx + 16 * i][e]); }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            acc[i][j] = fmaf(q[i].x, k4[j].x, acc[i][j]);
            acc[i][j] = fmaf(q[i].y, k4[j].y, acc[i][j]);
            acc[i][j] = fmaf(q[i].z, k4[j].z, acc[i][j]);
            acc[i][j] = fmaf(q[i].w, k4[j].w, acc[i][j]);
          }
      }
    }
    float* out = p.cb + (slot * p.G + job) * (int64_t)CP * CP;      // [t][s]
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) out[(ty * 4 + i) * CP + tx + 16 * j] = acc[i][j];
    return;
  }
  const int h = blockIdx.y / (tiles_n * tiles_v), tile = blockIdx.y % (tiles_n * tiles_v);
  const int e0 = (tile / tiles_v) * TP, c0 = (tile % tiles_v) * TP;
  const int g = h / (p.H / p.G);
  float4 bv[CP / 16], xv[CP / 16];
  {
    const float* r = p.xbc + (int64_t)t0 * ch;
#pragma unroll
    for (int k = 0; k < CP / 16; ++k) {
      const int s = ls + 16 * k;
      bv[k] = load4<VEC>(r + (int64_t)s * ch + inner + g * p.N + e0 + le, s < n ? p.N - e0 - le : 0);
      xv[k] = load4<VEC>(r + (int64_t)s * ch + h * p.Pd + c0 + le, s < n ? p.Pd - c0 - le : 0);
    }
  }
  if (tid < 32) chunk_log_decay(p.la + (int64_t)t0 * p.H + h, p.H, n, cum);
  __syncthreads();
  if (tid < CP) wgt[tid] = tid < n ? (float)exp(cum[n - 1] - cum[tid]) * p.dt[(int64_t)(t0 + tid) * p.H + h] : 0.f;
  if (tile == 0 && tid == 0) p.decay[slot * p.H + h] = (float)exp(cum[n - 1]);
  __syncthreads();
#pragma unroll
  for (int k = 0; k < CP / 16; ++k) {
    const float w = wgt[ls + 16 * k];
    put4(&a_s[ls + 16 * k][le], bv[k]);
    put4(&b_s[ls + 16 * k][le], make_float4(xv[k].x * w, xv[k].y * w, xv[k].z * w, xv[k].w * w));
  }
  __syncthreads();
#pragma unroll 8
  for (int s = 0; s < n; ++s) {
    const float4 a = get4(&a_s[s][ty * 4]), w = get4(&b_s[s][tx * 4]);
    const float av[4] = {a.x, a.y, a.z, a.w}, wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
  }
  float* U = p.U + (slot * p.H + h) * (int64_t)p.N * p.Pd;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int e = e0 + ty * 4 + i, x = c0 + tx * 4;
    if (e < p.N) store4<VEC>(U + (int64_t)e * p.Pd + x, p.Pd - x, acc[i]);
  }
}

// per V neighbouring elements of S: walk the request's chunks and leave in U's place the S that the chunk starts from;
// grid (elements / V / THREADS, B).  Eight chunks' loads are in flight, the next eight ahead of the last ones' stores.
template <int V>
__global__ void __launch_bounds__(THREADS) ssm_scan_kernel(const Params p) {
  constexpr int DEPTH = 8;
  pdl_enter();
  const int b = blockIdx.y;
  const int64_t per_head = (int64_t)p.N * p.Pd, total = per_head * p.H;
  const int64_t i = ((int64_t)blockIdx.x * THREADS + threadIdx.x) * V;
  const int t_begin = p.cu[b], len = p.cu[b + 1] - t_begin;
  if (i >= total || len <= 1) return;
  const int h = (int)(i / per_head);
  float* S_g = p.state + (int64_t)p.slots[b] * p.ld_state + i;
  Vec<V> S;
#pragma unroll
  for (int e = 0; e < V; ++e) S.x[e] = 0.f;
  if (!p.fresh[b]) S = ldv<V>(S_g);
  const int64_t slot0 = chunk_slot(t_begin, b, 0);
  float* U = p.U + slot0 * total + i;
  const float* dec = p.decay + slot0 * p.H + h;
  const int chunks = (len + CP - 1) / CP;
  Vec<V> u[DEPTH], nxt[DEPTH];
#pragma unroll
  for (int j = 0; j < DEPTH; ++j)
    if (j < chunks) u[j] = ldv<V>(U + (int64_t)j * total);
  for (int c = 0; c < chunks; c += DEPTH) {
#pragma unroll
    for (int j = 0; j < DEPTH; ++j)
      if (c + DEPTH + j < chunks) nxt[j] = ldv<V>(U + (int64_t)(c + DEPTH + j) * total);
#pragma unroll
    for (int j = 0; j < DEPTH; ++j) {
      if (c + j < chunks) {
        stv<V>(U + (int64_t)(c + j) * total, S);
        const float d = dec[(int64_t)(c + j) * p.H];
#pragma unroll
        for (int e = 0; e < V; ++e) S.x[e] = fmaf(S.x[e], d, u[j].x[e]);
      }
    }
#pragma unroll
    for (int j = 0; j < DEPTH; ++j) u[j] = nxt[j];
  }
  stv<V>(S_g, S);
}

// y for one (chunk, head, 64 value columns); grid (chunks, H * column tiles, B).  The passes over the state's channels load
// the next pass's tiles into registers while they compute.
template <bool VEC>
__global__ void __launch_bounds__(THREADS, 3) ssm_outputs_kernel(const Params p) {
  constexpr int LDC = KT + 4;
  __shared__ __align__(16) float tiles[CP * LDT];
  static_assert(CP * LDC + KT * TP <= CP * LDT, "a pass's tiles fit where A lies afterwards");
  float (*C_s)[LDC] = reinterpret_cast<float (*)[LDC]>(tiles);                   // [token][state channel]
  float (*S_s)[TP] = reinterpret_cast<float (*)[TP]>(tiles + CP * LDC);          // [state channel][value column]
  float (*A_s)[LDT] = reinterpret_cast<float (*)[LDT]>(tiles);                   // [token t][token s], after the passes
  __shared__ __align__(16) float x_s[CP][TP];      // [token s][value column]
  __shared__ double cum[CP];
  __shared__ float dts[CP];
  pdl_enter();
  const int tiles_v = (p.Pd + TP - 1) / TP;
  const int b = blockIdx.z, c = blockIdx.x, h = blockIdx.y / tiles_v, c0 = (blockIdx.y % tiles_v) * TP;
  const int t_begin = p.cu[b], t_end = p.cu[b + 1];
  const int t0 = t_begin + c * CP;
  if (t_end - t_begin <= 1 || t0 >= t_end) return;
  const int n = min(CP, t_end - t0), tid = threadIdx.x, ch = p.channels(), inner = p.inner();
  const int ty = tid >> 4, tx = tid & 15, g = h / (p.H / p.G);
  const int64_t slot = chunk_slot(t_begin, b, c);
  const float* S_prev = p.U + (slot * p.H + h) * (int64_t)p.N * p.Pd + c0;
  const float* Cp = p.xbc + (int64_t)t0 * ch + inner + (p.G + g) * p.N;
  // what this thread loads of a pass: C rows ct + 32 k at channels ce .., S rows (channels) sr + 16 k at columns sx ..
  const int ct = tid >> 3, ce = (tid & 7) * 4, sr = tid >> 4, sx = (tid & 15) * 4;
  float4 cv[CP / 32], sv[KT / 16];
  auto fetch = [&](int e0) {
#pragma unroll
    for (int k = 0; k < CP / 32; ++k)
      cv[k] = load4<VEC>(Cp + (int64_t)(ct + 32 * k) * ch + e0 + ce, ct + 32 * k < n ? p.N - e0 - ce : 0);
#pragma unroll
    for (int k = 0; k < KT / 16; ++k)
      sv[k] = load4<VEC>(S_prev + (int64_t)(e0 + sr + 16 * k) * p.Pd + sx, e0 + sr + 16 * k < p.N ? p.Pd - c0 - sx : 0);
  };
  fetch(0);
#pragma unroll
  for (int k = 0; k < CP / 16; ++k) {
    const int s = sr + 16 * k;
    put4(&x_s[s][sx], load4<VEC>(p.xbc + (int64_t)(t0 + s) * ch + h * p.Pd + c0 + sx, s < n ? p.Pd - c0 - sx : 0));
  }
  if (tid < 32) chunk_log_decay(p.la + (int64_t)t0 * p.H + h, p.H, n, cum);
  if (tid < CP) dts[tid] = tid < n ? p.dt[(int64_t)(t0 + tid) * p.H + h] : 0.f;
  float r[4][4] = {};
  for (int e0 = 0; e0 < p.N; e0 += KT) {
    __syncthreads();                               // the last pass is done with the tiles
#pragma unroll
    for (int k = 0; k < CP / 32; ++k) put4(&C_s[ct + 32 * k][ce], cv[k]);
#pragma unroll
    for (int k = 0; k < KT / 16; ++k) put4(&S_s[sr + 16 * k][sx], sv[k]);
    __syncthreads();
    if (e0 + KT < p.N) fetch(e0 + KT);
#pragma unroll 2
    for (int e = 0; e < KT; e += 4) {
      float4 q[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) q[i] = get4(&C_s[ty * 4 + i][e]);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float4 s4 = get4(&S_s[e + u][tx * 4]);
        const float sw[4] = {s4.x, s4.y, s4.z, s4.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float qv = u == 0 ? q[i].x : u == 1 ? q[i].y : u == 2 ? q[i].z : q[i].w;
#pragma unroll
          for (int j = 0; j < 4; ++j) r[i][j] = fmaf(qv, sw[j], r[i][j]);
        }
      }
    }
  }
  __syncthreads();
  // A[t][s] = (C_t . B_s) exp(c_t - c_s) dt_s for s <= t; r <- exp(c_t) r, which the sums over s then join
  const float* cb = p.cb + (slot * p.G + g) * (int64_t)CP * CP;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i;
    const float4 v = get4(cb + t * CP + tx * 4);
    const float vv[4] = {v.x, v.y, v.z, v.w};
    float a[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = tx * 4 + j;
      a[j] = (s <= t && t < n) ? vv[j] * expf((float)(cum[t] - cum[s])) * dts[s] : 0.f;
    }
    put4(&A_s[t][tx * 4], make_float4(a[0], a[1], a[2], a[3]));
    const float d = expf((float)cum[t]);
#pragma unroll
    for (int j = 0; j < 4; ++j) r[i][j] *= d;
  }
  __syncthreads();
  const int last = min(ty * 4 + 3, n - 1);         // (A is zero beyond t, x_s beyond the chunk's tokens)
  for (int s = 0; s <= last; s += 4) {
    float4 q[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) q[i] = get4(&A_s[ty * 4 + i][s]);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const float4 x4 = get4(&x_s[s + u][tx * 4]);
      const float xw[4] = {x4.x, x4.y, x4.z, x4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float qv = u == 0 ? q[i].x : u == 1 ? q[i].y : u == 2 ? q[i].z : q[i].w;
#pragma unroll
        for (int j = 0; j < 4; ++j) r[i][j] = fmaf(qv, xw[j], r[i][j]);
      }
    }
  }
  const float D = p.D[h];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty * 4 + i;
    if (t >= n) continue;
    const float4 x4 = get4(&x_s[t][tx * 4]);
    const float o[4] = {fmaf(D, x4.x, r[i][0]), fmaf(D, x4.y, r[i][1]), fmaf(D, x4.z, r[i][2]), fmaf(D, x4.w, r[i][3])};
    store4<VEC>(p.y + (int64_t)(t0 + t) * inner + (int64_t)h * p.Pd + c0 + tx * 4, p.Pd - c0 - tx * 4, o);
  }
}

// ---------------------------------------------------------------- gate, norm, the convolution's inputs
constexpr int POST_THREADS = 128;
constexpr int HOLD = 4;                             // runs a thread holds in registers (longer parts read theirs again)

// The last CTAs of the launch: run `job` of the channels of a request (V channels a thread).  Four rows at a time are read
// before they are written; rows rise, so a row is read before it is overwritten.
template <int V>
__device__ __forceinline__ void move_inputs(const Params& p, int job, int jobs_per_request) {
  const int b = job / jobs_per_request;
  const int start = p.cu[b], n = p.cu[b + 1] - start, rows = p.taps - 1, ch = p.channels();
  const int c = ((job % jobs_per_request) * POST_THREADS + threadIdx.x) * V;
  if (n <= 0 || c >= ch) return;
  float* hist = p.state + (int64_t)p.slots[b] * p.ld_state + p.hist + c;
  const float* x = p.P + (int64_t)start * p.ldp + p.inner() + c;
  const bool have = !p.fresh[b];
  for (int r0 = 0; r0 < rows; r0 += 4) {
    Vec<V> v[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int i = n - rows + r0 + u;              // index inside the portion; negative: from the inputs before it
#pragma unroll
      for (int e = 0; e < V; ++e) v[u].x[e] = 0.f;
      if (r0 + u >= rows) continue;
      if (i >= 0) v[u] = ldv<V>(x + (int64_t)i * p.ldp);
      else if (have) v[u] = ldv<V>(hist + (int64_t)(rows + i) * ch);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (r0 + u < rows) stv<V>(hist + (int64_t)(r0 + u) * ch, v[u]);
  }
}

// W threads (a warp, or the whole CTA) share a part of a token's row: rows_ctas CTAs of POST_THREADS / W parts each, then
// the CTAs that move the convolution's inputs.  out: rows of stride ldo, columns [inner, pad_to) are filled with zeros.
template <typename TO, int V, int W>
__global__ void __launch_bounds__(POST_THREADS)
ssm_post_kernel(const Params p, const float* __restrict__ weight, float eps, int parts, TO* __restrict__ out, int64_t ldo,
                int pad_to, int rows_ctas, int jobs_per_request) {
  __shared__ float red[33];
  pdl_enter();
  if ((int)blockIdx.x >= rows_ctas) return move_inputs<V>(p, blockIdx.x - rows_ctas, jobs_per_request);
  const int inner = p.inner(), len = inner / parts, tid = threadIdx.x % W;
  const int64_t job = (int64_t)blockIdx.x * (POST_THREADS / W) + threadIdx.x / W;
  if (job >= (int64_t)p.T * parts) return;           // (a whole warp of them, or the CTA: W divides it)
  const int t = (int)(job / parts), part = (int)(job % parts);
  const float* y = p.y + (int64_t)t * inner + (int64_t)part * len;
  const float* z = p.P + (int64_t)t * p.ldp + (int64_t)part * len;
  auto gated = [&](const Vec<V>& a, const Vec<V>& g) {
    Vec<V> v;
#pragma unroll
    for (int e = 0; e < V; ++e) v.x[e] = a.x[e] * silu_f(g.x[e]);
    return v;
  };
  Vec<V> hold[HOLD], gate[HOLD];
#pragma unroll
  for (int k = 0; k < HOLD; ++k) {
    const int i = (k * W + tid) * V;
    if (i < len) { hold[k] = ldv<V>(y + i); gate[k] = ldv<V>(z + i); }
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < HOLD; ++k) {
    if ((k * W + tid) * V >= len) continue;
    hold[k] = gated(hold[k], gate[k]);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(hold[k].x[e], hold[k].x[e], ss);
  }
  for (int i = (HOLD * W + tid) * V; i < len; i += W * V) {
    const Vec<V> v = gated(ldv<V>(y + i), ldv<V>(z + i));
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v.x[e], v.x[e], ss);
  }
  ss = W == 32 ? warp_sum(ss) : block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / (float)len + eps);
  TO* o = out + (int64_t)t * ldo + (int64_t)part * len;
  const float* w = weight + (int64_t)part * len;
  auto put = [&](int i, const Vec<V>& v) {
    const Vec<V> wv = ldv<V>(w + i);
    if constexpr (V == 4 && sizeof(TO) == 2) {
      uint2 u;
      __nv_bfloat162* hh = reinterpret_cast<__nv_bfloat162*>(&u);
      hh[0] = __floats2bfloat162_rn(v.x[0] * inv * wv.x[0], v.x[1] * inv * wv.x[1]);
      hh[1] = __floats2bfloat162_rn(v.x[2] * inv * wv.x[2], v.x[3] * inv * wv.x[3]);
      *reinterpret_cast<uint2*>(o + i) = u;
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) o[i + e] = from_f32<TO>(v.x[e] * inv * wv.x[e]);
    }
  };
#pragma unroll
  for (int k = 0; k < HOLD; ++k) {
    const int i = (k * W + tid) * V;
    if (i < len) put(i, hold[k]);
  }
  for (int i = (HOLD * W + tid) * V; i < len; i += W * V) put(i, gated(ldv<V>(y + i), ldv<V>(z + i)));
  if (part == parts - 1)
    for (int i = inner + tid; i < pad_to; i += W) out[(int64_t)t * ldo + i] = from_f32<TO>(0.f);
}

template <int V, int L>
void launch_step(const Params& p, cudaStream_t stream) {
  constexpr int PT = V * L, R = THREADS / L;
  const dim3 grid((p.Pd + PT - 1) / PT, p.H, p.B);
  const size_t smem = sizeof(float) * ((size_t)2 * p.N + PT + (THREADS / 32) * PT);
  const int rpt = (p.N + R - 1) / R;
  if (rpt <= 4) launch_pdl(ssm_step_kernel<V, L, 4>, grid, dim3(THREADS), smem, stream, p);
  else if (rpt <= 8) launch_pdl(ssm_step_kernel<V, L, 8>, grid, dim3(THREADS), smem, stream, p);
  else if (rpt <= 16) launch_pdl(ssm_step_kernel<V, L, 16>, grid, dim3(THREADS), smem, stream, p);
  else launch_pdl(ssm_step_kernel<V, L, 0>, grid, dim3(THREADS), smem, stream, p);
}

template <int V>
void launch_prep(const Params& p, cudaStream_t stream) {
  const dim3 grid((p.T + PREP_TOKENS - 1) / PREP_TOKENS, (p.channels() + PREP_THREADS * V - 1) / (PREP_THREADS * V) + 1);
  switch (p.taps) {
    case 1: launch_pdl(ssm_prep_kernel<V, 1>, grid, dim3(PREP_THREADS), 0, stream, p); break;
    case 2: launch_pdl(ssm_prep_kernel<V, 2>, grid, dim3(PREP_THREADS), 0, stream, p); break;
    case 3: launch_pdl(ssm_prep_kernel<V, 3>, grid, dim3(PREP_THREADS), 0, stream, p); break;
    case 4: launch_pdl(ssm_prep_kernel<V, 4>, grid, dim3(PREP_THREADS), 0, stream, p); break;
    default: launch_pdl(ssm_prep_kernel<V, 0>, grid, dim3(PREP_THREADS), 0, stream, p);
  }
}

bool al16(const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; }

}  // namespace

DINFER_DEFINE_LAST_ERROR()

// Floats of work space that a step of T tokens in B requests needs for its portions (0 where every request brings one).
DINFER_API int64_t dinfer_state_space_work_floats(int64_t T, int B, int H, int G, int N, int P) {
  const int64_t slots = T / CP + B, channels = (int64_t)H * P + 2 * (int64_t)G * N;
  auto r4 = [](int64_t n) { return (n + 3) / 4 * 4; };
  return r4(T * channels) + 2 * r4(T * H) + slots * H * (int64_t)N * P + r4(slots * H) + slots * G * CP * CP + 4;
}

// The recurrence of a step.  proj: f32 rows [z | x | B | C | dt] of stride ldp; conv_w [channels, taps], conv_b [channels],
// dt_bias, A_log, D [H] f32; state: f32 rows of stride ld_state, S [H, N, P] first, the convolution's (taps - 1) inputs
// [taps - 1, channels] from `hist` on (only read here: dinfer_state_space_post moves them on); cu [B + 1], slots, fresh [B];
// y [T, H * P] f32.  single / portions: whether some request brings exactly one token / more than one; max_q_len: a bound
// of the longest portion; work: dinfer_state_space_work_floats() floats, 16-byte aligned (null without portions).
DINFER_API int dinfer_state_space(const float* proj, int64_t ldp, const float* conv_w, const float* conv_b,
                                  const float* dt_bias, const float* A_log, const float* D, float* state, int64_t ld_state,
                                  int hist, const int* cu, const int* slots, const int* fresh, float* y, float* work, int T,
                                  int B, int H, int G, int N, int P, int taps, int single, int portions, int max_q_len,
                                  cudaStream_t stream) {
  if (T < 0 || B <= 0 || H <= 0 || G <= 0 || H % G || N <= 0 || P <= 0 || taps <= 0 || B > 65535)
    return refuse(DINFER_BAD_ARGUMENT, "state_space: bad sizes T=%d B=%d H=%d G=%d N=%d P=%d taps=%d", T, B, H, G, N, P, taps);
  Params p{};
  p.P = proj; p.ldp = ldp; p.conv_w = conv_w; p.conv_b = conv_b; p.dt_bias = dt_bias; p.A_log = A_log; p.D = D;
  p.state = state; p.ld_state = ld_state; p.hist = hist; p.cu = cu; p.slots = slots; p.fresh = fresh; p.y = y;
  p.T = T; p.B = B; p.H = H; p.G = G; p.N = N; p.Pd = P; p.taps = taps;
  const int64_t size = (int64_t)H * N * P;
  const int ch = p.channels(), inner = p.inner();
  if (ldp < (int64_t)inner + ch + H || hist < size || ld_state < hist + (int64_t)(taps - 1) * ch)
    return refuse(DINFER_BAD_ARGUMENT, "state_space: a row stride is shorter than its row");
  const int tiles_n = (N + TP - 1) / TP, tiles_v = (P + TP - 1) / TP;
  if (H > 65535 || (int64_t)H * tiles_n * tiles_v + G > 65535) return refuse(DINFER_BAD_ARGUMENT, "state_space: too many tiles for the grid");
  if (sizeof(float) * (size_t)(2 * N + 9 * 64) > 48 * 1024) return refuse(DINFER_BAD_ARGUMENT, "state_space: %d state channels are too many", N);
  if (T == 0) return 0;
  const bool state_vec = P % 4 == 0 && ld_state % 4 == 0 && al16(state);
  if (single) {
    if (!state_vec) launch_step<1, 32>(p, stream);
    else if (P <= 16) launch_step<4, 4>(p, stream);
    else if (P <= 32) launch_step<4, 8>(p, stream);
    else launch_step<4, 16>(p, stream);
  }
  if (portions) {
    if (!work || !al16(work) || max_q_len <= 0) return refuse(DINFER_BAD_ARGUMENT, "state_space: portions need work space and their longest");
    const int chunks = (max_q_len + CP - 1) / CP;
    const int64_t chunk_slots = (int64_t)T / CP + B;
    auto r4 = [](int64_t n) { return (n + 3) / 4 * 4; };
    p.U = work;
    p.cb = p.U + chunk_slots * size;
    if ((chunk_slots * size) % 4) p.cb += 4 - (chunk_slots * size) % 4;
    p.xbc = p.cb + chunk_slots * G * CP * CP;
    p.dt = p.xbc + r4((int64_t)T * ch);
    p.la = p.dt + r4((int64_t)T * H);
    p.decay = p.la + r4((int64_t)T * H);
    if (ch % 4 == 0 && ldp % 4 == 0 && inner % 4 == 0 && al16(proj)) launch_prep<4>(p, stream);
    else launch_prep<1>(p, stream);
    // 16-byte loads of the convolved rows, of the states and of y: every width and base allows them
    const bool vec = P % 4 == 0 && N % 4 == 0 && al16(y);
    launch_pdl(vec ? ssm_sums_kernel<true> : ssm_sums_kernel<false>, dim3(chunks, H * tiles_n * tiles_v + G, B), dim3(THREADS), 0, stream, p);
    if (state_vec) launch_pdl(ssm_scan_kernel<4>, dim3((unsigned)((size / 4 + THREADS - 1) / THREADS), B), dim3(THREADS), 0, stream, p);
    else launch_pdl(ssm_scan_kernel<1>, dim3((unsigned)((size + THREADS - 1) / THREADS), B), dim3(THREADS), 0, stream, p);
    launch_pdl(vec ? ssm_outputs_kernel<true> : ssm_outputs_kernel<false>, dim3(chunks, H * tiles_v, B), dim3(THREADS), 0, stream, p);
  }
  return cuda_status("state_space");
}

// out[t] = y[t] * silu(z[t]), each of `parts` equal parts of the row divided by its root mean square, times weight [H * P];
// out: rows of stride ldo, columns [H * P, pad_to) get zeros.  Then every request's last (taps - 1) convolution inputs
// become its state's.
DINFER_API int dinfer_state_space_post(const float* y, const float* proj, int64_t ldp, const float* weight, float eps,
                                       int parts, void* out, int64_t ldo, int pad_to, float* state, int64_t ld_state,
                                       int hist, const int* cu, const int* slots, const int* fresh, int T, int B, int H,
                                       int G, int N, int P, int taps, int out_dtype, cudaStream_t stream) {
  if (T < 0 || B <= 0 || H <= 0 || G <= 0 || N <= 0 || P <= 0 || taps <= 0 || parts <= 0 || ((int64_t)H * P) % parts)
    return refuse(DINFER_BAD_ARGUMENT, "state_space_post: bad sizes T=%d B=%d H=%d P=%d parts=%d", T, B, H, P, parts);
  Params p{};
  p.P = proj; p.ldp = ldp; p.state = state; p.ld_state = ld_state; p.hist = hist; p.cu = cu; p.slots = slots;
  p.fresh = fresh; p.y = const_cast<float*>(y); p.T = T; p.B = B; p.H = H; p.G = G; p.N = N; p.Pd = P; p.taps = taps;
  const int inner = p.inner(), len = inner / parts;
  if (ldp < (int64_t)inner + p.channels() || ldo < (pad_to > inner ? pad_to : inner) || ld_state < hist + (int64_t)(taps - 1) * p.channels())
    return refuse(DINFER_BAD_ARGUMENT, "state_space_post: a row stride is shorter than its row");
  if ((int64_t)T * parts + (int64_t)B * p.channels() > 0x7fffffffLL) return refuse(DINFER_BAD_ARGUMENT, "state_space_post: too many rows for the grid");
  if (T == 0) return 0;
  const bool vec = len % 4 == 0 && p.channels() % 4 == 0 && hist % 4 == 0 && ld_state % 4 == 0 && ldp % 4 == 0 && ldo % 4 == 0 &&
                   al16(state) && al16(y) && al16(proj) && al16(weight) && al16(out);
  // parts that a warp can hold go a warp each (unless there are too few of them to fill the device)
  const bool warps = len <= 32 * HOLD * (vec ? 4 : 1) && (int64_t)T * parts >= 592;
  const int per = warps ? POST_THREADS / 32 : 1;
  const int rows_ctas = (int)(((int64_t)T * parts + per - 1) / per);
  const int run = POST_THREADS * (vec ? 4 : 1), jobs = taps > 1 ? (p.channels() + run - 1) / run : 0;
  const dim3 grid((unsigned)(rows_ctas + (int64_t)B * jobs));
#define GO(V, W) launch_pdl(ssm_post_kernel<TO, V, W>, grid, dim3(POST_THREADS), 0, stream, p, weight, eps, parts, (TO*)out, \
                            ldo, pad_to, rows_ctas, jobs)
  DINFER_DISPATCH_DTYPE(out_dtype, TO, {
    if (vec) { if (warps) GO(4, 32); else GO(4, POST_THREADS); }
    else { if (warps) GO(1, 32); else GO(1, POST_THREADS); }
    return cuda_status("state_space_post");
  });
#undef GO
  return 0;
}
