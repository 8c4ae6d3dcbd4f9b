// build: precise-math
// Ragged-batch kernels for decoders whose residual is a small set of parallel streams ("hyper-connections"): a sublayer reads a weighted sum of
// the streams, and its output joins all of them while they are mixed with one another.
//
//   stream_mix_norm   per token row, one pass:
//                       v   = scale * (y + bias)                               the finished sublayer's output (fp32 from here on)
//                       x_t = sum_s mix[s, t] x_s + w_out[t] v                 all streams at once from the old ones
//                       u   = sum_s w_in[s] x_s                                what the next sublayer reads
//                       out = u / sqrt(mean(u^2) + eps) * gamma                in the activation dtype
//
// Each part is optional: without y the streams stay as they are, without gamma nothing is read.  Streams, sums, statistic and weights are fp32
// whatever the activation dtype is.  At the start of a model all streams are equal: they are then given as ONE row per token and written as
// separate rows by the first sublayer's join.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "../common/host.h"

namespace dsb {
namespace hyper {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

struct alignas(8) bf16x4 { __nv_bfloat162 a, b; };
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const bf16x4 v = *reinterpret_cast<const bf16x4*>(p);
  const float2 lo = __bfloat1622float2(v.a), hi = __bfloat1622float2(v.b);
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  bf16x4 o;
  o.a = __floats2bfloat162_rn(v.x, v.y);
  o.b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<bf16x4*>(p) = o;
}
__device__ __forceinline__ void axpy(float4& d, float a, float4 v) {
  d.x = fmaf(a, v.x, d.x);
  d.y = fmaf(a, v.y, d.y);
  d.z = fmaf(a, v.z, d.z);
  d.w = fmaf(a, v.w, d.w);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// sum over the block (called once per kernel); every thread gets the result.  `red` holds 32 floats.
__device__ __forceinline__ float block_sum(float v, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  return warp_sum(t);
}

struct MixArgs {
  const float* x;       // [T, S, dim], or [T, dim] when `shared_row`: the streams before the join
  float* x_out;         // [T, S, dim]: the streams after it (may be x itself; null: not written)
  const float* bias;    // [dim] or null
  const float* scale;   // [dim] or null
  const float* mix;     // [S, S]: mix[s * S + t] carries stream s into stream t
  const float* w_out;   // [S]
  const float* w_in;    // [S] or null: ones
  const float* gamma;   // [dim] or null
  const int* rows;      // output row r works on token row rows[r]; null: r
  long long y_ld;       // elements between the rows of y
  int shared_row;
  int S, dim;
  float eps;
};

// One block per row.  ST streams (compile time), 16-byte accesses (dim a multiple of 4, aligned bases), a thread keeps the V vectors of u it owns
// in registers between the statistic and the scaling: dim <= 4 * V * blockDim.
template <typename TY, typename TO, int ST, int V>
__global__ void stream_mix_norm_vec_kernel(const MixArgs a, const TY* __restrict__ y, TO* __restrict__ out) {
  __shared__ float red[32];
  const int r = blockIdx.x, src = a.rows ? a.rows[r] : r, nv = a.dim >> 2;
  const float* x = a.x + static_cast<size_t>(src) * a.dim * (a.shared_row ? 1 : ST);
  float mix[ST][ST], wo[ST], wi[ST];
  if (y != nullptr) {
#pragma unroll
    for (int s = 0; s < ST; ++s) {
      wo[s] = a.w_out[s];
#pragma unroll
      for (int t = 0; t < ST; ++t) mix[s][t] = a.mix[s * ST + t];
    }
  }
#pragma unroll
  for (int s = 0; s < ST; ++s) wi[s] = a.w_in ? a.w_in[s] : 1.f;
  float4 u[V];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const int c = 4 * (threadIdx.x + i * blockDim.x);
    u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < 4 * nv) {
      float4 xs[ST];
      if (a.shared_row) {
        const float4 v = load4(x + c);
#pragma unroll
        for (int s = 0; s < ST; ++s) xs[s] = v;
      } else {
#pragma unroll
        for (int s = 0; s < ST; ++s) xs[s] = load4(x + static_cast<size_t>(s) * a.dim + c);
      }
      if (y != nullptr) {
        float4 v = load4(y + static_cast<size_t>(src) * a.y_ld + c);
        if (a.bias) { const float4 b = load4(a.bias + c); v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w; }
        if (a.scale) { const float4 m = load4(a.scale + c); v.x *= m.x; v.y *= m.y; v.z *= m.z; v.w *= m.w; }
        float4 n[ST];
#pragma unroll
        for (int t = 0; t < ST; ++t) {
          n[t] = make_float4(wo[t] * v.x, wo[t] * v.y, wo[t] * v.z, wo[t] * v.w);
#pragma unroll
          for (int s = 0; s < ST; ++s) axpy(n[t], mix[s][t], xs[s]);
          if (a.x_out) store4(a.x_out + (static_cast<size_t>(src) * ST + t) * a.dim + c, n[t]);
        }
#pragma unroll
        for (int t = 0; t < ST; ++t) axpy(u[i], wi[t], n[t]);
      } else {
#pragma unroll
        for (int s = 0; s < ST; ++s) axpy(u[i], wi[s], xs[s]);
      }
      ss += u[i].x * u[i].x + u[i].y * u[i].y + u[i].z * u[i].z + u[i].w * u[i].w;
    }
  }
  if (a.gamma == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(a.dim) + a.eps);
  TO* o = out + static_cast<size_t>(r) * a.dim;
#pragma unroll
  for (int i = 0; i < V; ++i) {
    const int c = 4 * (threadIdx.x + i * blockDim.x);
    if (c < 4 * nv) {
      const float4 g = load4(a.gamma + c);
      store4(o + c, make_float4(u[i].x * inv * g.x, u[i].y * inv * g.y, u[i].z * inv * g.z, u[i].w * inv * g.w));
    }
  }
}

// Any number of streams, any width.  Shared memory: S floats per thread (the old streams of the entry it works on; no other thread touches
// them), then dim floats (the row u, written and read back by the same thread).
template <typename TY, typename TO>
__global__ void stream_mix_norm_kernel(const MixArgs a, const TY* __restrict__ y, TO* __restrict__ out) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  const int r = blockIdx.x, src = a.rows ? a.rows[r] : r, S = a.S;
  const float* x = a.x + static_cast<size_t>(src) * a.dim * (a.shared_row ? 1 : S);
  float* xs = sm + threadIdx.x;  // xs[s * blockDim.x]
  float* ubuf = sm + S * blockDim.x;
  float ss = 0.f;
  for (int c = threadIdx.x; c < a.dim; c += blockDim.x) {
    for (int s = 0; s < S; ++s) xs[s * blockDim.x] = a.shared_row ? x[c] : x[static_cast<size_t>(s) * a.dim + c];
    float v = 0.f, u = 0.f;
    if (y != nullptr) {
      v = to_f(y[static_cast<size_t>(src) * a.y_ld + c]);
      if (a.bias) v += a.bias[c];
      if (a.scale) v *= a.scale[c];
    }
    for (int t = 0; t < S; ++t) {
      float n = xs[t * blockDim.x];
      if (y != nullptr) {
        n = a.w_out[t] * v;
        for (int s = 0; s < S; ++s) n = fmaf(a.mix[s * S + t], xs[s * blockDim.x], n);
        if (a.x_out) a.x_out[(static_cast<size_t>(src) * S + t) * a.dim + c] = n;
      }
      u = fmaf(a.w_in ? a.w_in[t] : 1.f, n, u);
    }
    ubuf[c] = u;
    ss += u * u;
  }
  if (a.gamma == nullptr) return;
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(a.dim) + a.eps);
  for (int c = threadIdx.x; c < a.dim; c += blockDim.x) out[static_cast<size_t>(r) * a.dim + c] = from_f<TO>(ubuf[c] * inv * a.gamma[c]);
}

template <typename TY, typename TO>
static int launch(const MixArgs& a, const void* y, void* out, long long n, bool vec, cudaStream_t stream) {
  const unsigned grid = static_cast<unsigned>(n);
  const TY* yy = static_cast<const TY*>(y);
  TO* oo = static_cast<TO*>(out);
  if (vec) {
    const int nv = a.dim / 4;
    const int threads = nv >= 1024 ? 512 : (nv >= 256 ? 256 : (nv >= 96 ? 128 : 64));
    const bool wide = nv > 2 * threads;
#define GO(ST)                                                                                                \
  do {                                                                                                        \
    if (wide) stream_mix_norm_vec_kernel<TY, TO, ST, 4><<<grid, threads, 0, stream>>>(a, yy, oo);             \
    else stream_mix_norm_vec_kernel<TY, TO, ST, 2><<<grid, threads, 0, stream>>>(a, yy, oo);                  \
  } while (0)
    switch (a.S) {
      case 1: GO(1); break;
      case 2: GO(2); break;
      case 3: GO(3); break;
      default: GO(4); break;
    }
#undef GO
  } else {
    const int threads = 128;
    const size_t smem = (static_cast<size_t>(a.S) * threads + a.dim) * sizeof(float);
    auto kern = stream_mix_norm_kernel<TY, TO>;
    DSB_REQUIRE(smem <= 200 * 1024, "stream_mix_norm: %d streams of width %d", a.S, a.dim);
    if (smem > 40 * 1024) DSB_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
    kern<<<grid, threads, smem, stream>>>(a, yy, oo);
  }
  DSB_CHECK_CUDA(cudaGetLastError());
  return DSB_OK;
}

}  // namespace hyper
}  // namespace dsb

// x fp32: the streams [T, S, dim], or (shared_row) one row [T, dim] that stands for all of them.  y (null: no join) [T, y_ld] in y_dtype (0 =
// bf16, 1 = fp32): the finished sublayer's output; bias, scale [dim] fp32 or null; mix [S, S] (from, to), w_out [S].  The joined streams go to
// x_out [T, S, dim] (x itself unless shared_row; null: nowhere).  gamma (null: nothing is read) [dim]: out [n, dim] in out_dtype receives the
// RMS-normed sum of the streams weighted with w_in [S] (null: ones).  rows (null, or n int32 token rows): only these rows are worked on; x_out
// must then be null.
DSB_EXPORT int dsb200_stream_mix_norm(const float* x, int shared_row, float* x_out, const void* y, long long y_ld, int y_dtype, const float* bias,
                                      const float* scale, const float* mix, const float* w_out, const float* w_in, const float* gamma, void* out,
                                      int out_dtype, const int* rows, long long n, int S, int dim, float eps, cudaStream_t stream) {
  using namespace dsb;
  using namespace dsb::hyper;
  if (n == 0) return DSB_OK;
  DSB_REQUIRE(x != nullptr && S >= 1 && dim >= 1, "stream_mix_norm: %d streams of width %d", S, dim);
  DSB_REQUIRE(y == nullptr || (mix != nullptr && w_out != nullptr && y_ld >= dim), "stream_mix_norm: a join wants its mixing weights (row stride %lld)", y_ld);
  DSB_REQUIRE(gamma == nullptr || out != nullptr, "stream_mix_norm: no output");
  DSB_REQUIRE(x_out == nullptr || (rows == nullptr && (!shared_row || x_out != x)), "stream_mix_norm: streams are written for whole batches, beside a shared row");
  const MixArgs a{x, x_out, bias, scale, mix, w_out, w_in, gamma, rows, y_ld, shared_row, S, dim, eps};
  auto al = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool vec = S <= 4 && dim % 4 == 0 && dim <= 4 * 4 * 512 && y_ld % 4 == 0 && al(x) && al(x_out) && al(y) && al(bias) && al(scale) && al(gamma) && al(out);
  if (y_dtype == 0 && out_dtype == 0) return launch<bf16, bf16>(a, y, out, n, vec, stream);
  if (y_dtype == 0) return launch<bf16, float>(a, y, out, n, vec, stream);
  if (out_dtype == 0) return launch<float, bf16>(a, y, out, n, vec, stream);
  return launch<float, float>(a, y, out, n, vec, stream);
}
