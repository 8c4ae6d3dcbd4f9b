// build: precise-math
// Ragged-batch kernels of state-space mixers with one decay per head (state-space duality): per head a state S of N x P numbers,
//   S_t = exp(la_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,      dt = softplus(.), la = -rate dt,
// with B and C shared by the heads of a group.  Batches are described as in recurrent_ops.cu: `seq_desc` (int4 per sequence: first row, new
// tokens, tokens seen before, state slot); a sequence whose first new token has position 0 starts from zero state whatever its slot holds.
//
//   ssd_prepare       the short causal convolution over x | B | C with bias and silu (rows of this step, rows of the state, zeros before the
//                     start), and per head dt and la
//   ssd_scan          the recurrence token by token, the state in registers (decode steps, short portions, fp32, any sizes)
//   gated_group_norm  out = rms-in-groups(y silu(z)) * w
//
// Steps, decays, state, read-out and norm are fp32 for bf16 and fp32 activations alike.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "../common/host.h"

namespace dsb {
namespace ssd {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

struct alignas(8) bf16x4 {
  __nv_bfloat162 a, b;
};
// V consecutive values (V = 1, or V = 4 from an address that is a multiple of four values)
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&o)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
  } else {
    o[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void load_v(const bf16* p, float (&o)[V]) {
  if constexpr (V == 4) {
    const bf16x4 v = *reinterpret_cast<const bf16x4*>(p);
    const float2 lo = __bfloat1622float2(v.a), hi = __bfloat1622float2(v.b);
    o[0] = lo.x; o[1] = lo.y; o[2] = hi.x; o[3] = hi.y;
  } else {
    o[0] = to_f(*p);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&o)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
  else *p = o[0];
}
template <int V>
__device__ __forceinline__ void store_v(bf16* p, const float (&o)[V]) {
  if constexpr (V == 4) {
    bf16x4 v;
    v.a = __floats2bfloat162_rn(o[0], o[1]);
    v.b = __floats2bfloat162_rn(o[2], o[3]);
    *reinterpret_cast<bf16x4*>(p) = v;
  } else {
    *p = from_f<bf16>(o[0]);
  }
}

// silu of an activation: full precision for fp32 results, the fast exponential and division where the result is rounded to bf16 anyway
template <typename T>
__device__ __forceinline__ float silu_t(float z) {
  if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
  else return z / (1.f + expf(-z));
}
__device__ __forceinline__ float softplusf_(float z) { return z > 20.f ? z : log1pf(expf(z)); }

// ------------------------------------------------------------------------------------------------------------------ prepare
// A thread owns V channels and walks `rows` consecutive rows of the batch (PREP_ROWS of them; one when there are few rows: decode steps); the taps - 1 rows in front of the current one stay in
// registers (TAPS > 0; TAPS = 0: any number of taps, every row read per tap).  When the walk enters another sequence -- or starts in the
// middle of one -- that window is filled from the rows of this step, the state, or zeros.
constexpr int PREP_ROWS = 8, PREP_THREADS = 128;
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(PREP_THREADS)
ssd_prepare_kernel(const T* __restrict__ proj, long long ld, int col0, int dt_col0, const float* __restrict__ w, const float* __restrict__ b,
                   const T* __restrict__ state, const int4* __restrict__ seq_desc, const int* __restrict__ tok_seq, const float* __restrict__ dt_bias,
                   const float* __restrict__ rate, T* __restrict__ xbc, float* __restrict__ dt, float* __restrict__ la, int n_tokens, int C, int H,
                   int taps, int conv_blocks, int rows) {
  const int t_begin = blockIdx.y * rows, t_end = min(n_tokens, t_begin + rows);
  if (static_cast<int>(blockIdx.x) >= conv_blocks) {  // the step sizes: one thread per (row, head)
    for (int i = (blockIdx.x - conv_blocks) * PREP_THREADS + threadIdx.x; i < (t_end - t_begin) * H; i += (gridDim.x - conv_blocks) * PREP_THREADS) {
      const int t = t_begin + i / H, h = i % H;
      const float s = softplusf_(to_f(proj[static_cast<long long>(t) * ld + dt_col0 + h]) + dt_bias[h]);
      dt[static_cast<size_t>(t) * H + h] = s;
      la[static_cast<size_t>(t) * H + h] = -rate[h] * s;
    }
    return;
  }
  const int c = (blockIdx.x * PREP_THREADS + threadIdx.x) * V;
  if (c >= C) return;
  const int n_taps = TAPS > 0 ? TAPS : taps;
  float bias[V];
  load_v<V>(b + c, bias);
  constexpr int W = TAPS > 1 ? TAPS - 1 : 1;
  float wt[TAPS > 0 ? TAPS : 1][V], win[W][V];  // win[j]: the row taps - 1 - j positions back
  if constexpr (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_v<V>(w + static_cast<size_t>(j) * C + c, wt[j]);
  }
  int seq = -1;
  int4 sd = make_int4(0, 0, 0, 0);
  // row `back` positions before new token i of the current sequence
  auto earlier = [&](int i, int back, float (&o)[V]) {
    const int ii = i - back;
    if (ii >= 0) {
      load_v<V>(proj + static_cast<long long>(sd.x + ii) * ld + col0 + c, o);
    } else if (sd.z + ii >= 0) {
      load_v<V>(state + (static_cast<size_t>(sd.w) * (n_taps - 1) + n_taps - 1 + ii) * C + c, o);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = 0.f;
    }
  };
  for (int t = t_begin; t < t_end; ++t) {
    const int s = tok_seq[t];
    if (s != seq) {
      seq = s;
      sd = seq_desc[s];
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < W; ++j) earlier(t - sd.x, W - j, win[j]);
      }
    }
    float cur[V], acc[V];
    load_v<V>(proj + static_cast<long long>(t) * ld + col0 + c, cur);
    if constexpr (TAPS > 0) {
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = 0.f;
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < W; ++j)
#pragma unroll
          for (int e = 0; e < V; ++e) acc[e] = fmaf(wt[j][e], win[j][e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = fmaf(wt[TAPS - 1][e], cur[e], acc[e]);
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
#pragma unroll
          for (int j = 0; j + 1 < W; ++j) win[j][e] = win[j + 1][e];
          win[W - 1][e] = cur[e];
        }
      }
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) acc[e] = 0.f;
      for (int j = 0; j < n_taps; ++j) {
        float u[V], ww[V];
        earlier(t - sd.x, n_taps - 1 - j, u);
        load_v<V>(w + static_cast<size_t>(j) * C + c, ww);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(ww[e], u[e], acc[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = silu_t<T>(acc[e] + bias[e]);
    store_v<V>(xbc + static_cast<size_t>(t) * C + c, acc);
  }
}

// ------------------------------------------------------------------------------------------------------------------ scan
// One block per (sequence, head, tile of PT columns).  TX threads cover the tile's columns (V each), TY = SCAN_THREADS / TX groups the rows:
// thread (tx, ty) keeps rows ty, ty + TY, ... (RPT of them) of its V columns in registers.  Tokens are staged SCAN_CHUNK at a time; a thread
// leaves its part of every token's read-out in shared memory and the block adds the TY parts after the chunk (no reduction per token).
// The state in memory is [slots, H, N, P], so that a warp reads whole stretches of a row.
//
// A decay close to 1 is applied as S + (exp(la) - 1) S: the rounding of exp(la) itself would act on a slowly fading state in the same direction
// thousands of times, that of expm1 is smaller by the factor 1 - exp(la).
constexpr int SCAN_THREADS = 256, SCAN_CHUNK = 8;
constexpr float SLOW_DECAY = -0.7f;
template <typename T, int V, int RPT>
__global__ void __launch_bounds__(SCAN_THREADS)
ssd_scan_kernel(const T* __restrict__ xbc, const float* __restrict__ dt, const float* __restrict__ la, const float* __restrict__ Dskip,
                const int4* __restrict__ seq_desc, float* __restrict__ state, float* __restrict__ out, int H, int G, int N, int P, int PT, int TX,
                int TY, int min_new, int max_new) {
  extern __shared__ __align__(16) float sm[];
  const int4 sd = seq_desc[blockIdx.x];
  if (sd.y < min_new || sd.y > max_new) return;  // sequences another kernel of the step takes
  const int h = blockIdx.y, p0 = blockIdx.z * PT, tid = threadIdx.x;
  const int g = h / (H / G), inner = H * P, C = inner + 2 * G * N;
  const int cols = min(PT, P - p0);
  float* bs = sm;                              // [chunk][N]    dt B
  float* cs = bs + SCAN_CHUNK * N;             // [chunk][N]
  float* xs = cs + SCAN_CHUNK * N;             // [chunk][PT]
  float* es = xs + SCAN_CHUNK * PT;            // [chunk]       decay
  float* part = es + SCAN_CHUNK;               // [chunk][TY][PT]
  const int tx = tid % TX, ty = tid / TX;
  const bool live = ty < TY && tx * V < cols;
  float S[RPT][V];
  float* gS = state + ((static_cast<size_t>(sd.w) * H + h) * N) * P + p0 + tx * V;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int n = ty + i * TY;
    if (live && n < N && sd.z > 0) {
      load_v<V>(gS + static_cast<size_t>(n) * P, S[i]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) S[i][e] = 0.f;
    }
  }
  const float dsk = Dskip[h];
  for (int t0 = 0; t0 < sd.y; t0 += SCAN_CHUNK) {
    const int cn = min(SCAN_CHUNK, sd.y - t0);
    for (int x = tid; x < cn * N; x += SCAN_THREADS) {
      const int tok = x / N, n = x - tok * N;
      const size_t t = static_cast<size_t>(sd.x + t0 + tok);
      const T* row = xbc + t * C + inner + g * N + n;
      bs[tok * N + n] = dt[t * H + h] * to_f(row[0]);
      cs[tok * N + n] = to_f(row[G * N]);
    }
    for (int x = tid; x < cn * cols; x += SCAN_THREADS) {
      const int tok = x / cols, p = x - tok * cols;
      xs[tok * PT + p] = to_f(xbc[static_cast<size_t>(sd.x + t0 + tok) * C + h * P + p0 + p]);
    }
    if (tid < cn) {
      const float l = la[static_cast<size_t>(sd.x + t0 + tid) * H + h];
      es[tid] = l > SLOW_DECAY ? expm1f(l) : fmaxf(expf(l), 1e-38f);  // what the walk below multiplies by; the sign tells which
    }
    __syncthreads();
    if (live) {
      for (int tok = 0; tok < cn; ++tok) {
        const float e = es[tok];
        float xv[V], acc[V];
        load_v<V>(xs + tok * PT + tx * V, xv);
#pragma unroll
        for (int k = 0; k < V; ++k) acc[k] = 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
          const int n = ty + i * TY;
          if (n < N) {
            const float bb = bs[tok * N + n], cc = cs[tok * N + n];
#pragma unroll
            for (int k = 0; k < V; ++k) {
              S[i][k] = fmaf(e, S[i][k], e > 0.f ? bb * xv[k] : fmaf(bb, xv[k], S[i][k]));
              acc[k] = fmaf(cc, S[i][k], acc[k]);
            }
          }
        }
        store_v<V>(part + (tok * TY + ty) * PT + tx * V, acc);
      }
    }
    __syncthreads();
    for (int x = tid; x < cn * cols; x += SCAN_THREADS) {
      const int tok = x / cols, p = x - tok * cols;
      float y = dsk * xs[tok * PT + p];
      for (int r = 0; r < TY; ++r) y += part[(tok * TY + r) * PT + p];
      out[static_cast<size_t>(sd.x + t0 + tok) * inner + h * P + p0 + p] = y;
    }
    __syncthreads();
  }
  if (live) {
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int n = ty + i * TY;
      if (n < N) store_v<V>(gS + static_cast<size_t>(n) * P, S[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------------------------ gate and norm
// One block per (row, part): v = y silu(z) over the part's `per` values, out = v / sqrt(mean(v^2) + eps) * w.  Up to GN_KEEP V-vectors of a
// thread stay in registers between the statistic and the scaling; a wider part forms the rest twice.
constexpr int GN_THREADS = 256, GN_KEEP = 8;
template <typename T, int V>
__global__ void __launch_bounds__(GN_THREADS)
gated_group_norm_kernel(const float* __restrict__ y, const T* __restrict__ z, long long z_ld, const float* __restrict__ w, T* __restrict__ out,
                        long long out_ld, int per, int inner, float eps) {
  __shared__ float red[GN_THREADS / 32 + 1];
  const int t = blockIdx.x, c0 = blockIdx.y * per, n = per / V, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const float* yr = y + static_cast<size_t>(t) * inner + c0;
  const T* zr = z + static_cast<long long>(t) * z_ld + c0;
  auto gated = [&](int i, float (&o)[V]) {
    float a[V], b[V];
    load_v<V>(yr + i * V, a);
    load_v<V>(zr + i * V, b);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = a[e] * silu_t<T>(b[e]);
  };
  float keep[GN_KEEP][V], ss = 0.f;
#pragma unroll
  for (int k = 0; k < GN_KEEP; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n) {
      gated(i, keep[k]);
#pragma unroll
      for (int e = 0; e < V; ++e) ss += keep[k][e] * keep[k][e];
    }
  }
  for (int i = threadIdx.x + GN_KEEP * blockDim.x; i < n; i += blockDim.x) {
    float v[V];
    gated(i, v);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += v[e] * v[e];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int i = 0; i < static_cast<int>(blockDim.x >> 5); ++i) ss += red[i];
  const float inv = 1.f / sqrtf(ss / static_cast<float>(per) + eps);
  T* orow = out + static_cast<long long>(t) * out_ld + c0;
  auto emit = [&](int i, const float (&v)[V]) {
    float g[V], o[V];
    load_v<V>(w + c0 + i * V, g);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = v[e] * inv * g[e];
    store_v<V>(orow + i * V, o);
  };
#pragma unroll
  for (int k = 0; k < GN_KEEP; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n) emit(i, keep[k]);
  }
  for (int i = threadIdx.x + GN_KEEP * blockDim.x; i < n; i += blockDim.x) {
    float v[V];
    gated(i, v);
    emit(i, v);
  }
}

}  // namespace ssd
}  // namespace dsb

using namespace dsb;
using namespace dsb::ssd;

static inline bool mult4(long long v) { return v % 4 == 0; }
static inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// proj [T, ld] (dtype 0 = bf16, 1 = fp32) holds per token C channels (x | B | C of the recurrence) from col0 and H step-size pre-activations
// from dt_col0.  xbc [T, C] = silu(b + sum_j w[j, :] u_(t - taps + 1 + j)) with w fp32 [taps, C], b fp32 [C]; rows before this step come from
// state [slots, taps - 1, C] (null when taps = 1), rows before the sequence are zeros.  dt [T, H] = softplus(pre + dt_bias), la [T, H] = -rate dt
// (fp32).  Update the state afterwards with dsb200_conv_state_update.
DSB_EXPORT int dsb200_ssd_prepare(const void* proj, long long ld, int col0, int dt_col0, const float* w, const float* b, const void* state,
                                  const int* seq_desc, const int* tok_seq, const float* dt_bias, const float* rate, void* xbc, float* dt, float* la,
                                  int n_tokens, int C, int H, int taps, int dtype, cudaStream_t stream) {
  if (n_tokens == 0) return DSB_OK;
  DSB_REQUIRE(C >= 1 && H >= 1 && taps >= 1 && (taps == 1 || state != nullptr), "ssd_prepare: %d channels, %d heads, %d taps", C, H, taps);
  const bool vec = mult4(C) && mult4(ld) && mult4(col0) && al16(proj) && al16(w) && al16(b) && al16(state) && al16(xbc);
  const int V = vec ? 4 : 1;
  const int rows = n_tokens <= 512 ? 1 : PREP_ROWS;
  const int conv_blocks = (C / V + PREP_THREADS - 1) / PREP_THREADS, dt_blocks = (H * rows + PREP_THREADS - 1) / PREP_THREADS;
  const dim3 grid(conv_blocks + (dt_blocks < 4 ? dt_blocks : 4), (n_tokens + rows - 1) / rows);
#define LAUNCH(T, VV, TT)                                                                                                                              \
  ssd_prepare_kernel<T, VV, TT><<<grid, PREP_THREADS, 0, stream>>>((const T*)proj, ld, col0, dt_col0, w, b, (const T*)state, (const int4*)seq_desc, tok_seq, \
                                                                   dt_bias, rate, (T*)xbc, dt, la, n_tokens, C, H, taps, conv_blocks, rows)
#define BY_TAPS(T, VV)                       \
  do {                                       \
    if (taps == 2) LAUNCH(T, VV, 2);         \
    else if (taps == 3) LAUNCH(T, VV, 3);    \
    else if (taps == 4) LAUNCH(T, VV, 4);    \
    else LAUNCH(T, VV, 0);                   \
  } while (0)
  if (dtype == 0 && vec) BY_TAPS(bf16, 4);
  else if (dtype == 0) BY_TAPS(bf16, 1);
  else if (vec) BY_TAPS(float, 4);
  else BY_TAPS(float, 1);
#undef BY_TAPS
#undef LAUNCH
  DSB_CHECK_CUDA(cudaGetLastError());
  return DSB_OK;
}

// The recurrence over every sequence's new tokens in order, for the sequences that bring min_new .. max_new tokens.  xbc [T, H P + 2 G N]
// (x | B | C, head h reads group h / (H / G)), dt and la fp32 [T, H] as dsb200_ssd_prepare leaves them, Dskip fp32 [H]; state fp32
// [slots, H, N, P]; out fp32 [T, H P].  Any sizes with N <= 512 (1024 when P is a multiple of 4).
DSB_EXPORT int dsb200_ssd_scan(const void* xbc, const float* dt, const float* la, const float* Dskip, const int* seq_desc, float* state, float* out,
                               int n_seqs, int H, int G, int N, int P, int min_new, int max_new, int dtype, cudaStream_t stream) {
  if (n_seqs == 0) return DSB_OK;
  DSB_REQUIRE(H >= 1 && G >= 1 && H % G == 0 && N >= 1 && P >= 1, "ssd_scan: %d heads in %d groups, state %d x %d", H, G, N, P);
  const bool vec = mult4(P) && al16(state);
  const int V = vec ? 4 : 1, tile = vec ? 64 : 32;
  const int PT = P < tile ? P : tile, TX = (PT + V - 1) / V, TY = SCAN_THREADS / TX;
  const int need = (N + TY - 1) / TY;
  const int PTs = (PT + 3) / 4 * 4;  // columns of a staged row
  const size_t smem = (static_cast<size_t>(SCAN_CHUNK) * (2 * N + PTs + 1 + TY * PTs) + 8) * sizeof(float);
  DSB_REQUIRE(need <= 64 && smem <= 200 * 1024, "ssd_scan: a %d x %d state per head is not supported", N, P);
  const dim3 grid(n_seqs, H, (P + PT - 1) / PT);
  DSB_REQUIRE(PTs == PT || !vec, "ssd_scan: tile of %d columns", PT);
#define LAUNCH(T, VV, R)                                                                                                                        \
  do {                                                                                                                                          \
    if (smem > 48 * 1024) DSB_CHECK_CUDA(cudaFuncSetAttribute(ssd_scan_kernel<T, VV, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    ssd_scan_kernel<T, VV, R><<<grid, SCAN_THREADS, smem, stream>>>((const T*)xbc, dt, la, Dskip, (const int4*)seq_desc, state, out, H, G, N, P, PT, TX, TY, \
                                                                    min_new, max_new);                                                          \
  } while (0)
#define BY_ROWS(T, VV)                       \
  do {                                       \
    if (need <= 1) LAUNCH(T, VV, 1);         \
    else if (need <= 2) LAUNCH(T, VV, 2);    \
    else if (need <= 4) LAUNCH(T, VV, 4);    \
    else if (need <= 8) LAUNCH(T, VV, 8);    \
    else if (need <= 16) LAUNCH(T, VV, 16);  \
    else if (need <= 32) LAUNCH(T, VV, 32);  \
    else LAUNCH(T, VV, 64);                  \
  } while (0)
  if (dtype == 0 && vec) BY_ROWS(bf16, 4);
  else if (dtype == 0) BY_ROWS(bf16, 1);
  else if (vec) BY_ROWS(float, 4);
  else BY_ROWS(float, 1);
#undef BY_ROWS
#undef LAUNCH
  DSB_CHECK_CUDA(cudaGetLastError());
  return DSB_OK;
}

// out[t, :] = rms-in-groups(y[t, :] silu(z[t, :])) * w over `inner` values in `groups` equal consecutive parts (eps inside the root); y fp32
// [T, inner]; z [T, z_ld] and out [T, out_ld] in the activation dtype (0 = bf16, 1 = fp32), w fp32 [inner].
DSB_EXPORT int dsb200_gated_group_norm(const float* y, const void* z, long long z_ld, const float* w, void* out, long long out_ld, int n_tokens, int inner,
                                       int groups, float eps, int dtype, cudaStream_t stream) {
  if (n_tokens == 0) return DSB_OK;
  DSB_REQUIRE(groups >= 1 && groups <= 65535 && inner % groups == 0, "gated_group_norm: %d values do not split into %d equal parts", inner, groups);
  const int per = inner / groups;
  const bool vec = mult4(per) && mult4(z_ld) && mult4(out_ld) && al16(y) && al16(w) && (reinterpret_cast<uintptr_t>(z) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 7) == 0 &&
                   (dtype == 0 || al16(out));
  const int n = vec ? per / 4 : per;
  int block = 32;
  while (block < GN_THREADS && block * 2 < n) block *= 2;
  const dim3 grid(n_tokens, groups);
#define LAUNCH(T, VV) gated_group_norm_kernel<T, VV><<<grid, block, 0, stream>>>(y, (const T*)z, z_ld, w, (T*)out, out_ld, per, inner, eps)
  if (dtype == 0 && vec) LAUNCH(bf16, 4);
  else if (dtype == 0) LAUNCH(bf16, 1);
  else if (vec) LAUNCH(float, 4);
  else LAUNCH(float, 1);
#undef LAUNCH
  DSB_CHECK_CUDA(cudaGetLastError());
  return DSB_OK;
}
