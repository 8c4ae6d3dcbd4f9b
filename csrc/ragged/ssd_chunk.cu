// build: precise-math
// Chunk-parallel form of the state-space recurrence with one decay per head (see ssd_ops.cu) on tcgen05 tensor cores, for prompt portions.
// With a_i the running sum of la inside a chunk of 128 tokens and S the state in front of it,
//   y_i = sum_(j <= i) (C_i . B_j) exp(a_i - a_j) dt_j x_j  +  exp(a_i) C_i S  +  D x_i,
//   S'  = exp(a_last) S + sum_j B_j (exp(a_last - a_j) dt_j x_j)^T,
// four matrix products per chunk; only the chunk-to-chunk state is sequential.  One CTA walks the chunks of one (sequence, head):
//
//   warp 0      TMA producer (C | B, x tiles out of xbc [T, channels]) and the chunk's running sums: formed in double, kept as a pair of floats,
//               so that a_i - a_j keeps full fp32 accuracy however far the sum has run
//   warp 1      MMA issuer: G = C B^T;  Yc = C S;  dS = B^T X' (X'_j = exp(a_last - a_j) dt_j x_j);  Y = M x (M = the masked, decayed G, the
//               skip weight D on its diagonal)
//   warps 2-17  thread == (row, quarter of the columns): X' into shared memory, G -> M inside TMEM, the state in registers (fp32), outputs
//
// B, C and x are bf16 and enter as they are.  What is fp32 in the recurrence (M, X', S) enters the products as a sum of two bf16 numbers (16 bits
// of mantissa, two products each), accumulated in fp32; the state itself stays fp32 from chunk to chunk.
// Every wait is bounded: a role that gives up sets a flag that ends the others' waits, the copies in flight are waited for (bounded), TMEM is
// freed, an error word is written and the kernel returns.
#include "../common/host.h"
#include "../common/ptx.cuh"

namespace dsb {
namespace ssd {

constexpr int CQ = 128;                    // tokens per chunk
constexpr int CK_THREADS = 576;            // TMA warp, MMA warp, 16 compute warps
constexpr int CK_COMPUTE = 512;
constexpr int CK_CHUNK = 128 * 128;        // one [128 rows x 64 bf16] swizzled tile
constexpr long long CK_WAIT_CYCLES = 2000000000ll;

struct ChunkSmem {
  static constexpr int C_OFF = 0;                                  // [2 tiles]
  static constexpr int B_OFF = C_OFF + 2 * CK_CHUNK;               // [2 stages][2 tiles]
  static constexpr int X_OFF = B_OFF + 4 * CK_CHUNK;               // [2 stages][1 tile]
  static constexpr int XP_OFF = X_OFF + 2 * CK_CHUNK;              // X' high, low
  static constexpr int S_OFF = XP_OFF + 2 * CK_CHUNK;              // S high, low
  static constexpr int AR_OFF = S_OFF + 2 * CK_CHUNK;              // [2 stages][sum high | sum low | dt][128] floats
  static constexpr int BAR_OFF = AR_OFF + 2 * 3 * CQ * 4;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
};

struct ChunkParams {
  const float* dt;
  const float* la;
  const float* dskip;
  const int4* seq_desc;
  float* state;
  float* out;
  int* error;
  int H, G, N, P, min_new;
};

// true when the phase has completed; false when the wait gave up or another role did
__device__ __forceinline__ bool bounded_wait(uint64_t* bar, uint32_t parity, volatile int* quit) {
  bool ok = mbar_try_wait(bar, parity);
  if (!ok) {
    const long long t0 = clock64();
    while (!(ok = mbar_try_wait(bar, parity))) {
      if (*quit) break;
      if (clock64() - t0 > CK_WAIT_CYCLES) {
        *quit = 1;
        break;
      }
    }
  }
  return __all_sync(0xffffffffu, ok);  // one decision per warp: what follows is warp-wide
}

__global__ void __launch_bounds__(CK_THREADS, 1) ssd_chunk_kernel(const __grid_constant__ CUtensorMap tm_xbc, const ChunkParams p) {
  const int4 sd = p.seq_desc[blockIdx.y];
  if (sd.y < p.min_new) return;  // ssd_scan takes this sequence
  using SM = ChunkSmem;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + SM::BAR_OFF);
  uint64_t* bx_full = bars;        // [2]
  uint64_t* bx_empty = bars + 2;   // [2]
  uint64_t* sums_full = bars + 4;  // [2]
  uint64_t* c_full = bars + 6;
  uint64_t* c_empty = bars + 7;
  uint64_t* g_full = bars + 8;
  uint64_t* m_full = bars + 9;
  uint64_t* xp_full = bars + 10;
  uint64_t* s_full = bars + 11;
  uint64_t* ds_full = bars + 12;
  uint64_t* y_full = bars + 13;
  uint64_t* y_free = bars + 14;
  uint64_t* drained = bars + 15;
  uint32_t* tmem_ptr = reinterpret_cast<uint32_t*>(bars + 16);
  volatile int* quit = reinterpret_cast<volatile int*>(bars + 17);
  float* arrays = reinterpret_cast<float*>(smem + SM::AR_OFF);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.x, g = h / (p.H / p.G), N = p.N, P = p.P, inner = p.H * P;
  const int n_chunks = (sd.y + CQ - 1) / CQ;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tm_xbc);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&bx_full[i], 1);
      mbar_init(&bx_empty[i], 1);
      mbar_init(&sums_full[i], 1);
    }
    mbar_init(c_full, 1);
    mbar_init(c_empty, 1);
    mbar_init(g_full, 1);
    mbar_init(m_full, CK_COMPUTE);
    mbar_init(xp_full, CK_COMPUTE);
    mbar_init(s_full, CK_COMPUTE);
    mbar_init(ds_full, 1);
    mbar_init(y_full, 1);
    mbar_init(y_free, CK_COMPUTE);
    mbar_init(drained, 1);
    *quit = 0;
    fence_barrier_init();
  }
  if (warp == 1) {
    tmem_alloc<1>(tmem_ptr, 512);
    tmem_relinquish<1>();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = *tmem_ptr;
  const uint32_t TM_G = tm, TM_Y = tm + 128, TM_YC = tm + 192, TM_DS = tm + 256;

  int bx_sent = 0, c_sent = 0;  // loads issued (warp 0)
  if (warp == 0) {
    const int tiles = (N + 63) / 64;
    const int x_col = h * P, b_col = inner + g * N, c_col = inner + (p.G + g) * N;
    for (int c = 0; c < n_chunks; ++c) {
      const int st = c & 1, row0 = sd.x + c * CQ;
      if (!bounded_wait(&bx_empty[st], ((c >> 1) & 1) ^ 1, quit)) break;
      if (lane == 0) {
        mbar_expect_tx(&bx_full[st], (tiles + 1) * CK_CHUNK);
        for (int k = 0; k < tiles; ++k) tma_load_2d(&tm_xbc, &bx_full[st], smem + SM::B_OFF + (st * 2 + k) * CK_CHUNK, b_col + k * 64, row0);
        tma_load_2d(&tm_xbc, &bx_full[st], smem + SM::X_OFF + st * CK_CHUNK, x_col, row0);
      }
      ++bx_sent;
      // running sums of this chunk, four tokens per lane, in units of log2; tokens past the portion add nothing and have a step of 0
      float* ar = arrays + st * 3 * CQ;
      double a[4];
      float step[4];
      double run = 0.0;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = lane * 4 + e;
        const bool in = c * CQ + j < sd.y;
        const size_t at = static_cast<size_t>(row0 + j) * p.H + h;
        run += in ? static_cast<double>(p.la[at]) * 1.4426950408889634074 : 0.0;
        step[e] = in ? p.dt[at] : 0.f;
        a[e] = run;
      }
      double before = run;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double up = __shfl_up_sync(0xffffffffu, before, o);
        if (lane >= o) before += up;
      }
      before -= run;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const double s = before + a[e];
        const float hi = static_cast<float>(s);
        ar[lane * 4 + e] = hi;
        ar[CQ + lane * 4 + e] = static_cast<float>(s - static_cast<double>(hi));
        ar[2 * CQ + lane * 4 + e] = step[e];
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&sums_full[st]);
      if (!bounded_wait(c_empty, (c & 1) ^ 1, quit)) break;
      if (lane == 0) {
        mbar_expect_tx(c_full, tiles * CK_CHUNK);
        for (int k = 0; k < tiles; ++k) tma_load_2d(&tm_xbc, c_full, smem + SM::C_OFF + k * CK_CHUNK, c_col + k * 64, row0);
      }
      ++c_sent;
    }
  } else if (warp == 1) {
    const bool leader = elect_one();
    constexpr uint32_t idesc_g = umma_idesc(128, 128, 1, 1, 0, 0);                 // A = C rows, B = B rows (both K-major: K = state entry)
    // 64 columns whatever P is: a tile's columns past P hold other channels, their results are not read
    constexpr uint32_t idesc_y = umma_idesc(128, 64, 1, 1, 0, 1);                  // A = M (TMEM) or C, B = x or S (MN-major)
    constexpr uint32_t idesc_s = umma_idesc(128, 64, 1, 1, 1, 1);                  // A = B^T (MN-major), B = X' (MN-major)
    const uint32_t t0 = __shfl_sync(0xffffffffu, tm, 0);
    const uint64_t c_k = umma_smem_desc(smem_u32(smem + SM::C_OFF), 16, 1024);
    const uint64_t b_k = umma_smem_desc(smem_u32(smem + SM::B_OFF), 16, 1024);
    const uint64_t b_mn = umma_smem_desc(smem_u32(smem + SM::B_OFF), CK_CHUNK, 1024);
    const uint64_t x_mn = umma_smem_desc(smem_u32(smem + SM::X_OFF), CK_CHUNK, 1024);
    const uint64_t xp_mn = umma_smem_desc(smem_u32(smem + SM::XP_OFF), CK_CHUNK, 1024);
    const uint64_t s_mn = umma_smem_desc(smem_u32(smem + SM::S_OFF), CK_CHUNK, 1024);
    const int ks = N >> 4;
    for (int c = 0; c < n_chunks; ++c) {
      const int st = c & 1;
      const uint32_t b_off = static_cast<uint32_t>((st * 2 * CK_CHUNK) >> 4), x_off = static_cast<uint32_t>((st * CK_CHUNK) >> 4);
      if (!bounded_wait(&bx_full[st], (c >> 1) & 1, quit)) break;
      if (!bounded_wait(c_full, c & 1, quit)) break;
      tc_fence_after();
      if (leader) {  // the tensor pipe runs in issue order: the product before has read M out of these columns
        for (int kk = 0; kk < ks; ++kk) {
          const uint32_t o = static_cast<uint32_t>(((kk >> 2) * CK_CHUNK + (kk & 3) * 32) >> 4);
          umma_f16<1>(t0, c_k + o, b_k + b_off + o, idesc_g, kk != 0 ? 1u : 0u);
        }
        umma_commit<1>(g_full);
      }
      if (!bounded_wait(s_full, c & 1, quit)) break;
      if (c > 0 && !bounded_wait(y_free, (c - 1) & 1, quit)) break;
      tc_fence_after();
      if (leader) {
        for (int part = 0; part < 2; ++part)
          for (int kk = 0; kk < ks; ++kk)
            umma_f16<1>(t0 + 192, c_k + static_cast<uint32_t>(((kk >> 2) * CK_CHUNK + (kk & 3) * 32) >> 4),
                        s_mn + static_cast<uint32_t>((part * CK_CHUNK + kk * 2048) >> 4), idesc_y, (part | kk) != 0 ? 1u : 0u);
        umma_commit<1>(c_empty);
      }
      if (!bounded_wait(xp_full, c & 1, quit)) break;
      tc_fence_after();
      if (leader) {
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CQ / 16; ++kk)
            umma_f16<1>(t0 + 256, b_mn + b_off + static_cast<uint32_t>((kk * 2048) >> 4), xp_mn + static_cast<uint32_t>((part * CK_CHUNK + kk * 2048) >> 4),
                        idesc_s, (part | kk) != 0 ? 1u : 0u);
        umma_commit<1>(ds_full);
      }
      if (!bounded_wait(m_full, c & 1, quit)) break;
      tc_fence_after();
      if (leader) {
        for (int part = 0; part < 2; ++part)
#pragma unroll
          for (int kk = 0; kk < CQ / 16; ++kk)  // 16 tokens = 8 packed columns; the quarter that owns them keeps high | low in its 32 columns
            umma_f16_ts(t0 + 128, t0 + (kk >> 1) * 32 + part * 16 + (kk & 1) * 8, x_mn + x_off + static_cast<uint32_t>((kk * 2048) >> 4), idesc_y,
                        (part | kk) != 0 ? 1u : 0u);
        umma_commit<1>(y_full);
        umma_commit<1>(&bx_empty[st]);
      }
    }
  } else {
    const int q4 = warp & 3, part = (warp - 2) >> 2, row = q4 * 32 + lane, tid = threadIdx.x - 64;
    const uint32_t lane_off = static_cast<uint32_t>(q4 * 32) << 16;
    const int p0 = part * 16;                        // columns [p0, p0 + 16) of outputs and state
    const bool cols = p0 < P, rows = row < N;
    const float dsk = p.dskip[h];
    float* gS = p.state + ((static_cast<size_t>(sd.w) * p.H + h) * N + row) * P + p0;
    float S[16];
#pragma unroll
    for (int e = 0; e < 16; e += 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (cols && rows && sd.z > 0) v = *reinterpret_cast<const float4*>(gS + e);
      S[e] = v.x; S[e + 1] = v.y; S[e + 2] = v.z; S[e + 3] = v.w;
    }
    auto publish_state = [&]() {
      if (cols) {
        uint32_t hi[8], lo[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          hi[e] = pack_bf16x2(S[2 * e], S[2 * e + 1]);
          const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&hi[e]);
          lo[e] = pack_bf16x2(S[2 * e] - __low2float(hv), S[2 * e + 1] - __high2float(hv));
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          uint8_t* at = smem + SM::S_OFF + row * 128 + (((part * 2 + u) ^ (row & 7)) << 4);
          *reinterpret_cast<uint4*>(at) = make_uint4(hi[4 * u], hi[4 * u + 1], hi[4 * u + 2], hi[4 * u + 3]);
          *reinterpret_cast<uint4*>(at + CK_CHUNK) = make_uint4(lo[4 * u], lo[4 * u + 1], lo[4 * u + 2], lo[4 * u + 3]);
        }
      }
      fence_proxy_async_smem();
      mbar_arrive(s_full);
    };
    publish_state();
    bool done = true;
    for (int c = 0; c < n_chunks; ++c) {
      const int st = c & 1;
      const float* hi = arrays + st * 3 * CQ;
      const float* lo = hi + CQ;
      const float* step = lo + CQ;
      if (!bounded_wait(&sums_full[st], (c >> 1) & 1, quit) || !bounded_wait(&bx_full[st], (c >> 1) & 1, quit)) { done = false; break; }
      const float end_hi = hi[CQ - 1], end_lo = lo[CQ - 1];
      // X': 16-byte units of the x tile (8 per row)
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int id = tid + k * CK_COMPUTE, j = id >> 3, u = id & 7;
        const int at = j * 128 + ((u ^ (j & 7)) << 4);
        const uint4 xv = *reinterpret_cast<const uint4*>(smem + SM::X_OFF + st * CK_CHUNK + at);
        const float w = ex2_approx((end_hi - hi[j]) + (end_lo - lo[j])) * step[j];
        const uint32_t in[4] = {xv.x, xv.y, xv.z, xv.w};
        uint32_t oh[4], ol[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const __nv_bfloat162 xb = *reinterpret_cast<const __nv_bfloat162*>(&in[e]);
          const float a = w * __low2float(xb), b = w * __high2float(xb);
          oh[e] = pack_bf16x2(a, b);
          const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&oh[e]);
          ol[e] = pack_bf16x2(a - __low2float(hv), b - __high2float(hv));
        }
        *reinterpret_cast<uint4*>(smem + SM::XP_OFF + at) = make_uint4(oh[0], oh[1], oh[2], oh[3]);
        *reinterpret_cast<uint4*>(smem + SM::XP_OFF + CK_CHUNK + at) = make_uint4(ol[0], ol[1], ol[2], ol[3]);
      }
      fence_proxy_async_smem();
      mbar_arrive(xp_full);
      // G -> M, in the columns it came from: 32 tokens of the row -> 16 packed columns (high) + 16 (low)
      const float my_hi = hi[row], my_lo = lo[row];
      if (!bounded_wait(g_full, c & 1, quit)) { done = false; break; }
      tc_fence_after();
      {
        const uint32_t addr = TM_G + part * 32 + lane_off;
        const int j0 = part * 32;
        uint32_t ph[16], pl[16];
        if (j0 <= q4 * 32 + 31) {
          uint32_t gv[32];
          tmem_ld_32x32(addr, gv);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; e += 4) {
            const float4 ah = *reinterpret_cast<const float4*>(hi + j0 + e), al = *reinterpret_cast<const float4*>(lo + j0 + e),
                         as = *reinterpret_cast<const float4*>(step + j0 + e);
            const float jh[4] = {ah.x, ah.y, ah.z, ah.w}, jl[4] = {al.x, al.y, al.z, al.w}, js[4] = {as.x, as.y, as.z, as.w};
            float m[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              const int j = j0 + e + k;
              m[k] = __uint_as_float(gv[e + k]) * (ex2_approx((my_hi - jh[k]) + (my_lo - jl[k])) * js[k]);
              m[k] = j < row ? m[k] : (j == row ? m[k] + dsk : 0.f);
            }
#pragma unroll
            for (int k = 0; k < 4; k += 2) {
              const int o = (e + k) >> 1;
              ph[o] = pack_bf16x2(m[k], m[k + 1]);
              const __nv_bfloat162 hv = *reinterpret_cast<const __nv_bfloat162*>(&ph[o]);
              pl[o] = pack_bf16x2(m[k] - __low2float(hv), m[k + 1] - __high2float(hv));
            }
          }
        } else {  // every token of the quarter lies behind every row of the warp
#pragma unroll
          for (int e = 0; e < 16; ++e) ph[e] = pl[e] = 0u;
        }
        tmem_st_32x16(addr, ph);
        tmem_st_32x16(addr + 16, pl);
        tmem_st_wait();
      }
      tc_fence_before();
      mbar_arrive(m_full);
      // the state behind the chunk
      if (!bounded_wait(ds_full, c & 1, quit)) { done = false; break; }
      tc_fence_after();
      {
        uint32_t d[16];
        tmem_ld_32x16(TM_DS + p0 + lane_off, d);
        tmem_ld_wait();
        const float keep = ex2_approx(end_hi + end_lo);
#pragma unroll
        for (int e = 0; e < 16; ++e) S[e] = fmaf(keep, S[e], __uint_as_float(d[e]));
      }
      if (c + 1 < n_chunks) {
        tc_fence_before();
        publish_state();
      }
      if (!bounded_wait(y_full, c & 1, quit)) { done = false; break; }
      tc_fence_after();
      uint32_t y[16], yc[16];
      tmem_ld_32x16(TM_Y + p0 + lane_off, y);
      tmem_ld_32x16(TM_YC + p0 + lane_off, yc);
      tmem_ld_wait();
      tc_fence_before();
      mbar_arrive(y_free);
      const int i = c * CQ + row;
      if (cols && i < sd.y) {
        const float f = ex2_approx(my_hi + my_lo);
        float* dst = p.out + static_cast<size_t>(sd.x + i) * inner + h * P + p0;
#pragma unroll
        for (int e = 0; e < 16; e += 4)
          *reinterpret_cast<float4*>(dst + e) =
              make_float4(fmaf(f, __uint_as_float(yc[e]), __uint_as_float(y[e])), fmaf(f, __uint_as_float(yc[e + 1]), __uint_as_float(y[e + 1])),
                          fmaf(f, __uint_as_float(yc[e + 2]), __uint_as_float(y[e + 2])), fmaf(f, __uint_as_float(yc[e + 3]), __uint_as_float(y[e + 3])));
      }
    }
    if (done && cols && rows) {
#pragma unroll
      for (int e = 0; e < 16; e += 4) *reinterpret_cast<float4*>(gS + e) = make_float4(S[e], S[e + 1], S[e + 2], S[e + 3]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*quit) {  // copies and products in flight land before the CTA goes away
    volatile int never = 0;
    if (warp == 0) {
      for (int c = bx_sent > 2 ? bx_sent - 2 : 0; c < bx_sent; ++c) bounded_wait(&bx_full[c & 1], (c >> 1) & 1, &never);
      if (c_sent > 0) bounded_wait(c_full, (c_sent - 1) & 1, &never);
    } else if (warp == 1) {
      if (elect_one()) umma_commit<1>(drained);
      __syncwarp();
      bounded_wait(drained, 0, &never);
    }
    if (threadIdx.x == 0) *p.error = 1;
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc<1>(tm, 512);
  }
}

}  // namespace ssd
}  // namespace dsb

// The recurrence of dsb200_ssd_scan in its chunked form, for the sequences that bring at least min_new tokens (the others are left to
// dsb200_ssd_scan with max_new = min_new - 1).  xbc bf16 [T, H P + 2 G N], the rest as there; N a multiple of 16 up to 128, P a multiple of 16 up
// to 64, at least 64 channels, rows 16-byte aligned.  error: one int on the device, set to 1 when a wait inside the kernel gave up (the outputs are
// then incomplete); never cleared.
DSB_EXPORT int dsb200_ssd_chunk(const void* xbc, const float* dt, const float* la, const float* Dskip, const int* seq_desc, float* state, float* out,
                                int* error, int n_tokens, int n_seqs, int H, int G, int N, int P, int min_new, cudaStream_t stream) {
  using namespace dsb;
  using namespace dsb::ssd;
  if (n_seqs == 0 || n_tokens == 0) return DSB_OK;
  const int C = H * P + 2 * G * N;
  DSB_REQUIRE(H >= 1 && G >= 1 && H % G == 0 && N >= 16 && N <= 128 && N % 16 == 0 && P >= 16 && P <= 64 && P % 16 == 0 && C >= 64 && n_seqs <= 65535,
              "ssd_chunk: %d heads in %d groups, state %d x %d", H, G, N, P);
  DSB_REQUIRE(((reinterpret_cast<uintptr_t>(xbc) | reinterpret_cast<uintptr_t>(state) | reinterpret_cast<uintptr_t>(out)) & 15) == 0 && error != nullptr,
              "ssd_chunk: operands must be 16-byte aligned");
  CUtensorMap tm;
  const int rc = make_tensor_map_2d(&tm, TMA_BF16, xbc, n_tokens, C, C, CQ, 64, TMA_SW_128);
  if (rc) return rc;
  static bool attr_set = false;
  if (!attr_set) {
    DSB_CHECK_CUDA(cudaFuncSetAttribute(ssd_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, ChunkSmem::TOTAL));
    attr_set = true;
  }
  ChunkParams p{dt, la, Dskip, reinterpret_cast<const int4*>(seq_desc), state, out, error, H, G, N, P, min_new};
  ssd_chunk_kernel<<<dim3(H, n_seqs), CK_THREADS, ChunkSmem::TOTAL, stream>>>(tm, p);
  DSB_CHECK_CUDA(cudaGetLastError());
  return DSB_OK;
}
