// A state-space recurrence with one decay and one step size per token and head (Mamba-2's form).  Per head, with
// S [N][dv] in float, B and C vectors of N numbers shared by the heads of a group, x of dv:
//
//   dt_t = softplus(raw_t + dt_bias),   a_t = exp(-exp(A_log) dt_t)
//   S_t  = a_t S_{t-1} + dt_t B_t x_t^T,     y_t = S_t^T C_t + D x_t
//
// A mixer that makes its decays and weights itself (the gates of a matrix memory) brings them: log a_t as `logd`, the
// weight of B x^T in dt_t's place, no D.
//
// x, B and C arrive in the activation type as columns of one row per token (what a short convolution leaves), the raw
// step sizes as floats; step sizes, decays, state and sums are float.  The state of a sequence is its slot of the
// cache's state region ([slots][H][N][dv]): a step continues from it, whatever a prompt was cut into.
//
//   hb_ssd_scan      token by token, any sizes, both precisions: decoding, short steps, the 32-bit path
//   hb_ssd_chunked   prompts in bfloat16, 64 tokens at a time on the tensor cores, chunks side by side.  With
//                    L_t = sum of log decays from the chunk's start through t and S0 the state before the chunk:
//
//       y_t = e^{L_t} S0^T C_t + sum_{s <= t} e^{L_t - L_s} dt_s (C_t . B_s) x_s + D x_t
//       S0 of the next chunk = e^{L_last} S0 + sum_s e^{L_last - L_s} dt_s B_s x_s^T
//
//     in three launches: every chunk's own sum for the state; the states handed from chunk to chunk; the outputs.
//     B, C and x are exact bfloat16 operands.  What is float by nature (the state S0, the weighted x of the state's
//     sum, the weighted scores) enters the products as a high and a low bfloat16 part, so those products carry
//     about 16 bits of it.
#include "api.h"
#include "common.cuh"
#include "mma_utils.cuh"

struct SsdArgs {
  const void* xbc; int ld, b_off, c_off;      // row t: x at 0 [H][dv], B at b_off [G][N], C at c_off [G][N]
  const float* dt; int lddt;                  // raw step sizes [tokens][H]; with logd: the weights as they are
  const float* logd;                          // log decays [tokens][H] with dt's row stride, <= 0; null: from the step sizes
  const float* dt_bias; const float* a_log; const float* dskip;      // [H] each; null with logd
  float* state;                               // [slots][H][N][dv]
  const int* seq_slot; const int* seq_start;
  float* out; int ldo;                        // [tokens][H][dv]
  int H, G, N, dv;
  int cb;                                     // token by token: value channels per CTA (a power of two, at least 4)
  float* chunk_state; float* chunk_decay;     // chunked: [chunk][H][N][dv], [chunk][H]
  int vw;                                     // chunked: value channels per CTA, at most the kernel's DVM
};

__device__ __forceinline__ float ssd_softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// ---------------------------------------------------------------------------------------------
// Token by token.  A CTA owns cb value channels of one head of one sequence; a thread holds four neighbouring channels
// of RPT state rows in registers (rows tid / (cb / 4) + i * row groups), so a row of the state is read and written
// in runs of cb floats.  The row groups' parts of a token's read-out meet in shared memory after every SS_CHUNK tokens.
#define SS_THREADS 256
#define SS_CHUNK 8
template <typename T, int RPT>
__global__ void __launch_bounds__(SS_THREADS) ssd_scan_kernel(SsdArgs a) {
  extern __shared__ __align__(16) float sh[];
  const int ct = a.cb >> 2, rgs = SS_THREADS / ct, NP = rgs * RPT;
  float* Bs = sh;                                   // [SS_CHUNK][NP]
  float* Cs = Bs + SS_CHUNK * NP;                   // [SS_CHUNK][NP]
  float* xs = Cs + SS_CHUNK * NP;                   // [SS_CHUNK][cb]
  float4* red = reinterpret_cast<float4*>(xs + SS_CHUNK * a.cb);      // [SS_CHUNK][SS_THREADS]
  float* coef = reinterpret_cast<float*>(red + SS_CHUNK * SS_THREADS);   // [SS_CHUNK][2]: decay, step size
  pdl_wait();
  pdl_launch();
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int col0 = blockIdx.z * a.cb, c4 = (tid % ct) * 4, g = tid / ct;
  const int grp = h / (a.H / a.G);
  const int t0 = a.seq_start[b], t1 = a.seq_start[b + 1];
  float* S = a.state + (((size_t)a.seq_slot[b] * a.H + h) * a.N) * (size_t)a.dv;
  const bool vec = a.dv % 4 == 0;
  float s[RPT][4];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = g + i * rgs, c = col0 + c4;
    s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
    if (r < a.N && c < a.dv) {
      if (vec) {
        const float4 f = *reinterpret_cast<const float4*>(S + (size_t)r * a.dv + c);
        s[i][0] = f.x; s[i][1] = f.y; s[i][2] = f.z; s[i][3] = f.w;
      } else {
        for (int j = 0; j < 4; ++j)
          if (c + j < a.dv) s[i][j] = S[(size_t)r * a.dv + c + j];
      }
    }
  }
  for (int i = tid; i < SS_CHUNK * (2 * NP + a.cb); i += SS_THREADS) sh[i] = 0.0f;      // rows past N stay zero
  const bool given = a.logd != nullptr;
  const float neg_a = given ? 0.0f : -expf(a.a_log[h]), bias = given ? 0.0f : a.dt_bias[h], dskip = given ? 0.0f : a.dskip[h];
  for (int c0 = t0; c0 < t1; c0 += SS_CHUNK) {
    const int n = t1 - c0 < SS_CHUNK ? t1 - c0 : SS_CHUNK;
    __syncthreads();
    const T* base = (const T*)a.xbc + (size_t)c0 * a.ld;
    for (int i = tid; i < n * a.N; i += SS_THREADS) {
      const int tt = i / a.N, r = i - tt * a.N;
      const T* row = base + (size_t)tt * a.ld + (size_t)grp * a.N + r;
      Bs[tt * NP + r] = to_f32(row[a.b_off]);
      Cs[tt * NP + r] = to_f32(row[a.c_off]);
    }
    for (int i = tid; i < n * a.cb; i += SS_THREADS) {
      const int tt = i / a.cb, c = i - tt * a.cb;
      if (col0 + c < a.dv) xs[i] = to_f32(base[(size_t)tt * a.ld + (size_t)h * a.dv + col0 + c]);
    }
    if (tid < n) {
      const size_t at = (size_t)(c0 + tid) * a.lddt + h;
      const float dt = given ? a.dt[at] : ssd_softplus(a.dt[at] + bias);
      coef[2 * tid] = expf(given ? a.logd[at] : neg_a * dt);
      coef[2 * tid + 1] = dt;
    }
    __syncthreads();
    for (int tt = 0; tt < n; ++tt) {
      const float da = coef[2 * tt], dt = coef[2 * tt + 1];
      const float4 x = *reinterpret_cast<const float4*>(xs + tt * a.cb + c4);
      const float x0 = x.x * dt, x1 = x.y * dt, x2 = x.z * dt, x3 = x.w * dt;
      float o0 = 0.0f, o1 = 0.0f, o2 = 0.0f, o3 = 0.0f;
#pragma unroll
      for (int i = 0; i < RPT; ++i) {
        const float bv = Bs[tt * NP + g + i * rgs], cv = Cs[tt * NP + g + i * rgs];
        s[i][0] = fmaf(da, s[i][0], bv * x0); o0 = fmaf(s[i][0], cv, o0);
        s[i][1] = fmaf(da, s[i][1], bv * x1); o1 = fmaf(s[i][1], cv, o1);
        s[i][2] = fmaf(da, s[i][2], bv * x2); o2 = fmaf(s[i][2], cv, o2);
        s[i][3] = fmaf(da, s[i][3], bv * x3); o3 = fmaf(s[i][3], cv, o3);
      }
      red[tt * SS_THREADS + tid] = make_float4(o0, o1, o2, o3);
    }
    __syncthreads();
    for (int i = tid; i < n * a.cb; i += SS_THREADS) {
      const int tt = i / a.cb, c = i - tt * a.cb;
      if (col0 + c >= a.dv) continue;
      const float* p = reinterpret_cast<const float*>(red + tt * SS_THREADS) + c;
      float o = 0.0f;
      for (int k = 0; k < rgs; ++k) o += p[k * a.cb];
      a.out[(size_t)(c0 + tt) * a.ldo + (size_t)h * a.dv + col0 + c] = fmaf(dskip, xs[i], o);
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = g + i * rgs, c = col0 + c4;
    if (r < a.N && c < a.dv) {
      if (vec) {
        *reinterpret_cast<float4*>(S + (size_t)r * a.dv + c) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
      } else {
        for (int j = 0; j < 4; ++j)
          if (c + j < a.dv) S[(size_t)r * a.dv + c + j] = s[i][j];
      }
    }
  }
}

static int ssd_sms() {
  static int sms = 0;
  if (sms == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
  }
  return sms;
}

#define SS_CHECKS(name)                                                                                                       \
  HB_REQUIRE(n_seqs > 0 && heads > 0 && groups > 0 && N > 0 && dv > 0, name ": sizes must be positive");                       \
  HB_REQUIRE(heads % groups == 0, name ": %d heads are not a multiple of %d groups", heads, groups);                           \
  HB_REQUIRE(n_seqs <= 65535 && heads <= 65535, name ": too many sequences or heads");                                         \
  HB_REQUIRE(logd != nullptr || (dt_bias != nullptr && a_log != nullptr && dskip != nullptr),                                  \
             name ": needs log decays, or the step sizes' bias, the decay rates and D");                                       \
  HB_REQUIRE(((uintptr_t)state & 15) == 0, name ": the state must be 16-byte aligned")

extern "C" int hb_ssd_scan(int dtype, const void* xbc, int ld, int b_off, int c_off, const float* dt, int lddt,
                           const float* logd, const float* dt_bias, const float* a_log, const float* dskip, float* state, const int* seq_slot,
                           const int* seq_start, float* out, int ldo, int n_seqs, int heads, int groups, int N, int dv,
                           void* stream) {
  SS_CHECKS("ssd_scan");
  HB_REQUIRE(N <= 2048, "ssd_scan: %d state rows per head exceed the supported maximum 2048", N);
  int cb = 4;
  while (cb < 64 && cb < dv) cb <<= 1;
  while (cb > 4 && ceil_div(N, 1024 / cb) > 16) cb >>= 1;                                           // at most 16 rows a thread
  while (cb > 16 && (long long)n_seqs * heads * ceil_div(dv, cb) < 2LL * ssd_sms()) cb >>= 1;       // few CTAs: narrower ones
  const int rgs = 1024 / cb;
  const int need = ceil_div(N, rgs);
  const int rpt = need <= 1 ? 1 : need <= 2 ? 2 : need <= 4 ? 4 : need <= 8 ? 8 : 16;
  const size_t smem = (size_t)(SS_CHUNK * (2 * rgs * rpt + cb) + SS_CHUNK * SS_THREADS * 4 + 2 * SS_CHUNK) * sizeof(float);
  HB_REQUIRE(smem <= 220 * 1024 && ceil_div(dv, cb) <= 65535, "ssd_scan: %d state rows or %d value channels are too many", N, dv);
  const SsdArgs a{xbc, ld, b_off, c_off, dt, lddt, logd, dt_bias, a_log, dskip, state, seq_slot, seq_start, out, ldo, heads, groups, N, dv,
                  cb, nullptr, nullptr, 0};
  const dim3 grid(n_seqs, heads, ceil_div(dv, cb));
  cudaStream_t s = (cudaStream_t)stream;
#define SS_GO(T, RPT)                                                                                                          \
  do {                                                                                                                         \
    if (smem > 48 * 1024) cudaFuncSetAttribute(ssd_scan_kernel<T, RPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    hb_launch(ssd_scan_kernel<T, RPT>, grid, dim3(SS_THREADS), smem, s, a);                                                    \
  } while (0)
#define SS_GO_T(T)                                                                                                             \
  do {                                                                                                                         \
    if (rpt == 1) SS_GO(T, 1); else if (rpt == 2) SS_GO(T, 2); else if (rpt == 4) SS_GO(T, 4);                                  \
    else if (rpt == 8) SS_GO(T, 8); else SS_GO(T, 16);                                                                         \
  } while (0)
  if (dtype == HB_F32) SS_GO_T(float); else SS_GO_T(bf16);
#undef SS_GO_T
#undef SS_GO
  HB_CHECK_LAUNCH("ssd_scan");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Chunked form.  Chunk c of sequence b has index seq_start[b] / 64 + b + c in the scratch arrays: sequences' ranges do
// not meet, and floor(tokens / 64) + sequences bounds them all.  A CTA works on one chunk and up to SC_HEADS heads of one
// group, one after another: B (and C, and the scores) are the group's, what belongs to the next head is fetched while
// this one is computed.
#define SC_Q 64
#define SC_T 256
#define SC_HEADS 4
__device__ __forceinline__ int ssd_chunk_index(const SsdArgs& a, int b, int c) { return a.seq_start[b] / SC_Q + b + c; }

struct SsdTile {      // what a CTA of the chunked kernels works on
  int c, b, grp, h0, nh, v0, cols, tok0, n;
};
__device__ __forceinline__ bool ssd_tile(const SsdArgs& a, int vblocks, int hpc, SsdTile& w) {
  const int per = a.H / a.G, parts = (per + hpc - 1) / hpc;
  int y = blockIdx.y;
  w.c = blockIdx.x; w.b = blockIdx.z;
  w.v0 = (y % vblocks) * a.vw; y /= vblocks;
  w.grp = y / parts;
  const int part = y % parts;
  w.h0 = w.grp * per + part * hpc;
  w.nh = per - part * hpc < hpc ? per - part * hpc : hpc;
  w.cols = a.dv - w.v0 < a.vw ? a.dv - w.v0 : a.vw;
  const int t0 = a.seq_start[w.b], len = a.seq_start[w.b + 1] - t0;
  w.tok0 = t0 + w.c * SC_Q;
  w.n = len - w.c * SC_Q < SC_Q ? len - w.c * SC_Q : SC_Q;
  return w.n > 0;
}

// One warp: a chunk's step sizes and L_t (inclusive sums of log decays, to the base 2); tokens past the end get dt 0 and
// decay 1.
__device__ __forceinline__ void ssd_prepare(const SsdArgs& a, int h, int tok0, int n, float* dts, float* cum) {
  const int lane = threadIdx.x & 31;
  constexpr float LOG2E = 1.4426950408889634f;
  const size_t at = (size_t)(tok0 + 2 * lane) * a.lddt + h;
  const bool live0 = 2 * lane < n, live1 = 2 * lane + 1 < n;
  float d0 = 0.0f, d1 = 0.0f, l0 = 0.0f, l1 = 0.0f;
  if (a.logd != nullptr) {
    if (live0) { d0 = a.dt[at]; l0 = a.logd[at] * LOG2E; }
    if (live1) { d1 = a.dt[at + a.lddt]; l1 = a.logd[at + a.lddt] * LOG2E; }
  } else {
    const float neg_a = -expf(a.a_log[h]) * LOG2E, bias = a.dt_bias[h];
    if (live0) d0 = ssd_softplus(a.dt[at] + bias);
    if (live1) d1 = ssd_softplus(a.dt[at + a.lddt] + bias);
    l0 = neg_a * d0;
    l1 = neg_a * d1;
  }
  float run = l0 + l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += v;
  }
  dts[2 * lane] = d0; dts[2 * lane + 1] = d1;
  cum[2 * lane] = run - l1; cum[2 * lane + 1] = run;
}

// rows [64][cols] of bfloat16 from the token rows into shared memory [64][stride]; rows from n on and columns from
// `cols` to `padded` become zero.  vec: 16-byte pieces (columns and the row length multiples of 8, rows on 16 bytes).
__device__ __forceinline__ void ssd_load_rows(bf16* dst, int stride, const bf16* src, int ld, int n, int cols, int padded, bool vec) {
  const int per = padded >> 3;
  for (int i = threadIdx.x; i < SC_Q * per; i += SC_T) {
    const int r = i / per, c = (i - r * per) * 8;
    bf16* d = dst + r * stride + c;
    if (r < n && vec && c + 8 <= cols) {
      cp_async16(d, src + (size_t)r * ld + c);
    } else if (r >= n || c >= cols) {
      *reinterpret_cast<uint4*>(d) = make_uint4(0, 0, 0, 0);
    } else {
      for (int j = 0; j < 8; ++j) d[j] = c + j < cols ? src[(size_t)r * ld + c + j] : __float2bfloat16_rn(0.0f);
    }
  }
}

__device__ __forceinline__ float ssd_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ssd_split2(float x, float y, unsigned& hi, unsigned& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const unsigned*>(&h);
  lo = pack_bf16(x - f.x, y - f.y);
}

// A chunk's own contribution to the state: sum_s e^{L_last - L_s} dt_s B_s x_s^T, and its total decay.  A warp takes
// every eighth tile of 16 state rows.
template <int DVM>
__global__ void __launch_bounds__(SC_T) ssd_chunk_state_kernel(SsdArgs a, int vblocks, int vec, int hpc) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ __align__(16) float dts[SC_HEADS][SC_Q], cum[SC_HEADS][SC_Q];
  constexpr int XS = DVM + 8, PER = DVM / 8, PIECES = (SC_Q * PER + SC_T - 1) / SC_T;
  const int NP = (a.N + 15) & ~15, BS = NP + 8;
  bf16* Bs = reinterpret_cast<bf16*>(smem);          // [64][BS]
  bf16* Xh = Bs + SC_Q * BS;                         // [2][64][XS] weighted x, high parts
  bf16* Xl = Xh + 2 * SC_Q * XS;                     // low parts
  pdl_wait();
  pdl_launch();
  SsdTile w;
  if (!ssd_tile(a, vblocks, hpc, w)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bf16* rows = (const bf16*)a.xbc + (size_t)w.tok0 * a.ld;
  ssd_load_rows(Bs, BS, rows + a.b_off + (size_t)w.grp * a.N, a.ld, w.n, a.N, NP, vec);
  cp_async_commit();
  uint4 raw[PIECES];                                 // the next head's x, eight channels of a token a piece
  auto fetch = [&](int h) {
    const bf16* xr = rows + (size_t)h * a.dv + w.v0;
#pragma unroll
    for (int q = 0; q < PIECES; ++q) {
      const int i = threadIdx.x + q * SC_T, r = i / PER, c = (i % PER) * 8;
      raw[q] = make_uint4(0, 0, 0, 0);
      if (i >= SC_Q * PER || r >= w.n || c >= w.cols) continue;
      if (vec) {
        raw[q] = *reinterpret_cast<const uint4*>(xr + (size_t)r * a.ld + c);
      } else {
        bf16 v[8];
        for (int j = 0; j < 8; ++j) v[j] = c + j < w.cols ? xr[(size_t)r * a.ld + c + j] : __float2bfloat16_rn(0.0f);
        unsigned u[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const __nv_bfloat162 p = __halves2bfloat162(v[2 * j], v[2 * j + 1]);
          u[j] = *reinterpret_cast<const unsigned*>(&p);
        }
        raw[q] = make_uint4(u[0], u[1], u[2], u[3]);
      }
    }
  };
  fetch(w.h0);
  if (warp < w.nh) ssd_prepare(a, w.h0 + warp, w.tok0, w.n, dts[warp], cum[warp]);
  cp_async_wait<0>();
  __syncthreads();
  const size_t ci = ssd_chunk_index(a, w.b, w.c);
  const int mi = lane >> 3, l8 = lane & 7, g = lane >> 2, t = lane & 3;
  const bool pair = a.dv % 2 == 0;
  for (int ih = 0; ih < w.nh; ++ih) {
    const int h = w.h0 + ih;
    bf16* xh = Xh + (ih & 1) * SC_Q * XS;
    bf16* xl = Xl + (ih & 1) * SC_Q * XS;
    const float last = cum[ih][SC_Q - 1];
#pragma unroll
    for (int q = 0; q < PIECES; ++q) {
      const int i = threadIdx.x + q * SC_T, r = i / PER, c = (i % PER) * 8;
      if (i >= SC_Q * PER) continue;
      const float k = ssd_exp2(last - cum[ih][r]) * dts[ih][r];
      const unsigned u[4] = {raw[q].x, raw[q].y, raw[q].z, raw[q].w};
      unsigned hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u[j]));
        ssd_split2(f.x * k, f.y * k, hi[j], lo[j]);
      }
      *reinterpret_cast<uint4*>(xh + r * XS + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(xl + r * XS + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    if (ih + 1 < w.nh) fetch(h + 1);
    __syncthreads();      // also: the buffer written next was last read before the previous head's barrier
    float* out = a.chunk_state + ((ci * a.H + h) * a.N) * (size_t)a.dv + w.v0;
    if (threadIdx.x == 0 && w.v0 == 0) a.chunk_decay[ci * a.H + h] = ssd_exp2(last);
    for (int mt = warp; mt < NP / 16; mt += SC_T / 32) {
      float acc[DVM / 8][4];
#pragma unroll
      for (int i = 0; i < DVM / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
#pragma unroll
      for (int k = 0; k < SC_Q / 16; ++k) {
        unsigned a0, a1, a2, a3;
        ldmatrix_x4_trans(a0, a1, a2, a3, Bs + (k * 16 + (mi >> 1) * 8 + l8) * BS + mt * 16 + (mi & 1) * 8);
#pragma unroll
        for (int nd = 0; nd < DVM / 16; ++nd) {
          if (nd * 16 >= w.cols) continue;
          const int off = (k * 16 + (mi & 1) * 8 + l8) * XS + nd * 16 + (mi >> 1) * 8;
          unsigned b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, xh + off);
          mma16816(acc[2 * nd], a0, a1, a2, a3, b0, b1);
          mma16816(acc[2 * nd + 1], a0, a1, a2, a3, b2, b3);
          ldmatrix_x4_trans(b0, b1, b2, b3, xl + off);
          mma16816(acc[2 * nd], a0, a1, a2, a3, b0, b1);
          mma16816(acc[2 * nd + 1], a0, a1, a2, a3, b2, b3);
        }
      }
#pragma unroll
      for (int nd = 0; nd < DVM / 8; ++nd)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = mt * 16 + g + half * 8, v = nd * 8 + 2 * t;
          if (r >= a.N || v >= w.cols) continue;
          float* p = out + (size_t)r * a.dv + v;
          if (pair) *reinterpret_cast<float2*>(p) = make_float2(acc[nd][2 * half], acc[nd][2 * half + 1]);
          else {
            p[0] = acc[nd][2 * half];
            if (v + 1 < w.cols) p[1] = acc[nd][2 * half + 1];
          }
        }
    }
  }
}

// The states handed from chunk to chunk: what a chunk contributed is replaced by the state before it; the slot's state
// becomes the one after the step.  V neighbouring entries of a head's state per thread.  V = 8: the state before a chunk
// leaves as eight high and then eight low bfloat16 parts in the place of its eight floats, ready to be an operand.
template <int V>
__global__ void __launch_bounds__(128) ssd_state_pass_kernel(SsdArgs a) {
  pdl_wait();
  pdl_launch();
  const int b = blockIdx.z, h = blockIdx.y, per = a.N * a.dv;
  const int e = (blockIdx.x * 128 + threadIdx.x) * V;
  const int len = a.seq_start[b + 1] - a.seq_start[b], nc = (len + SC_Q - 1) / SC_Q;
  if (e >= per) return;
  float* S = a.state + ((size_t)a.seq_slot[b] * a.H + h) * per + e;
  const size_t c0 = ssd_chunk_index(a, b, 0);
  float* cs = a.chunk_state + (c0 * a.H + h) * per + e;
  const float* cd = a.chunk_decay + c0 * a.H + h;
  const size_t step = (size_t)a.H * per;
  float s[V];
  auto load = [&](float* v, const float* p) {
    if constexpr (V == 8) {
      const float4 f = *reinterpret_cast<const float4*>(p), k = *reinterpret_cast<const float4*>(p + 4);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; v[4] = k.x; v[5] = k.y; v[6] = k.z; v[7] = k.w;
    } else v[0] = p[0];
  };
  auto hand_on = [&](float* p, const float* v) {
    if constexpr (V == 8) {
      unsigned hi[4], lo[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) ssd_split2(v[2 * j], v[2 * j + 1], hi[j], lo[j]);
      reinterpret_cast<uint4*>(p)[0] = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      reinterpret_cast<uint4*>(p)[1] = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    } else p[0] = v[0];
  };
  load(s, S);
  for (int c = 0; c < nc; c += 4) {      // the loads of four chunks go ahead of their stores
    float x[4][V], d[4];
#pragma unroll
    for (int q = 0; q < 4; ++q)
      if (c + q < nc) { load(x[q], cs + (size_t)(c + q) * step); d[q] = cd[(size_t)(c + q) * a.H]; }
#pragma unroll
    for (int q = 0; q < 4; ++q)
      if (c + q < nc) {
        hand_on(cs + (size_t)(c + q) * step, s);
#pragma unroll
        for (int j = 0; j < V; ++j) s[j] = fmaf(d[q], s[j], x[q][j]);
      }
  }
  if constexpr (V == 8) {
    reinterpret_cast<float4*>(S)[0] = make_float4(s[0], s[1], s[2], s[3]);
    reinterpret_cast<float4*>(S)[1] = make_float4(s[4], s[5], s[6], s[7]);
  } else S[0] = s[0];
}

// The outputs of a chunk.  Warp w owns tokens 16 (w mod 4) .. and one half of the value channels.
template <int DVM>
__global__ void __launch_bounds__(SC_T) ssd_chunk_out_kernel(SsdArgs a, int vblocks, int vec, int hpc, int stages) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ __align__(16) float dts[SC_HEADS][SC_Q], cum[SC_HEADS][SC_Q];
  constexpr int XS = DVM + 8, HALF = DVM / 2;
  const int NP = (a.N + 15) & ~15, BS = NP + 8;
  bf16* Cs = reinterpret_cast<bf16*>(smem);          // [64][BS]
  bf16* Bs = Cs + SC_Q * BS;                         // [64][BS]
  bf16* ring = Bs + SC_Q * BS;                       // per stage: x [64][XS], the state's high and low parts [NP][XS] each
  const int stage_len = (SC_Q + 2 * NP) * XS;
  pdl_wait();
  pdl_launch();
  SsdTile w;
  if (!ssd_tile(a, vblocks, hpc, w)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bf16* rows = (const bf16*)a.xbc + (size_t)w.tok0 * a.ld;
  const size_t ci = ssd_chunk_index(a, w.b, w.c);
  const bool packed = a.dv % 8 == 0;                 // the states lie as high and low parts already
  auto stage = [&](int ih) {
    bf16* Xs = ring + (ih % stages) * stage_len;
    bf16* Sh = Xs + SC_Q * XS;
    bf16* Sl = Sh + NP * XS;
    const int h = w.h0 + ih;
    ssd_load_rows(Xs, XS, rows + (size_t)h * a.dv + w.v0, a.ld, w.n, w.cols, DVM, vec);
    const float* S0 = a.chunk_state + ((ci * a.H + h) * a.N) * (size_t)a.dv + w.v0;
    constexpr int PER = DVM / 8;
    for (int i = threadIdx.x; i < NP * PER; i += SC_T) {
      const int r = i / PER, v = (i % PER) * 8;
      bf16* dh = Sh + r * XS + v;
      bf16* dl = Sl + r * XS + v;
      const float* src = S0 + (size_t)r * a.dv + v;
      if (r >= a.N || v >= w.cols) {
        *reinterpret_cast<uint4*>(dh) = make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(dl) = make_uint4(0, 0, 0, 0);
      } else if (packed) {
        cp_async16(dh, src);
        cp_async16(dl, src + 4);
      } else {
        for (int j = 0; j < 8; j += 2) {
          const float f0 = v + j < w.cols ? src[j] : 0.0f, f1 = v + j + 1 < w.cols ? src[j + 1] : 0.0f;
          unsigned hi, lo;
          ssd_split2(f0, f1, hi, lo);
          *reinterpret_cast<unsigned*>(dh + j) = hi;
          *reinterpret_cast<unsigned*>(dl + j) = lo;
        }
      }
    }
    cp_async_commit();
  };
  ssd_load_rows(Cs, BS, rows + a.c_off + (size_t)w.grp * a.N, a.ld, w.n, a.N, NP, vec);
  ssd_load_rows(Bs, BS, rows + a.b_off + (size_t)w.grp * a.N, a.ld, w.n, a.N, NP, vec);
  stage(0);
  if (warp < w.nh) ssd_prepare(a, w.h0 + warp, w.tok0, w.n, dts[warp], cum[warp]);
  const int rb = warp & 3, cb = (warp >> 2) * HALF;
  const int mi = lane >> 3, l8 = lane & 7, g = lane >> 2, t = lane & 3;
  const int tr0 = rb * 16 + g, tr1 = tr0 + 8;
  const bool live = rb * 16 < w.n && cb < w.cols;    // a warp without tokens or channels keeps the barriers company
  const bool pair = a.dv % 2 == 0 && a.ldo % 2 == 0;
  float sc[8][4];                                    // C B^T of the warp's tokens: the group's, kept for all heads
  for (int ih = 0; ih < w.nh; ++ih) {
    if (stages > 1 && ih + 1 < w.nh) {
      stage(ih + 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (live) {
      if (ih == 0) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) sc[i][j] = 0.0f;
        for (int ks = 0; ks < NP / 16; ++ks) {
          unsigned a0, a1, a2, a3;
          ldmatrix_x4(a0, a1, a2, a3, Cs + (rb * 16 + (lane & 15)) * BS + ks * 16 + (lane >> 4) * 8);
#pragma unroll
          for (int np = 0; np < 4; ++np) {
            if (np > rb) continue;                   // keys after the warp's tokens
            unsigned b0, b1, b2, b3;
            ldmatrix_x4(b0, b1, b2, b3, Bs + (np * 16 + l8 + ((lane >> 4) << 3)) * BS + ks * 16 + ((lane >> 3) & 1) * 8);
            mma16816(sc[2 * np], a0, a1, a2, a3, b0, b1);
            mma16816(sc[2 * np + 1], a0, a1, a2, a3, b2, b3);
          }
        }
      }
      const int h = w.h0 + ih;
      const bf16* Xs = ring + (ih % stages) * stage_len;
      const bf16* Sh = Xs + SC_Q * XS;
      const bf16* Sl = Sh + NP * XS;
      float acc[HALF / 8][4];
#pragma unroll
      for (int i = 0; i < HALF / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
#pragma unroll 2
      for (int ks = 0; ks < NP / 16; ++ks) {         // C S0
        unsigned a0, a1, a2, a3;
        ldmatrix_x4(a0, a1, a2, a3, Cs + (rb * 16 + (lane & 15)) * BS + ks * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int nd = 0; nd < HALF / 16; ++nd) {
          const int off = (ks * 16 + (mi & 1) * 8 + l8) * XS + cb + nd * 16 + (mi >> 1) * 8;
          unsigned b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, Sh + off);
          mma16816(acc[2 * nd], a0, a1, a2, a3, b0, b1);
          mma16816(acc[2 * nd + 1], a0, a1, a2, a3, b2, b3);
          ldmatrix_x4_trans(b0, b1, b2, b3, Sl + off);
          mma16816(acc[2 * nd], a0, a1, a2, a3, b0, b1);
          mma16816(acc[2 * nd + 1], a0, a1, a2, a3, b2, b3);
        }
      }
      const float L0 = cum[ih][tr0], L1 = cum[ih][tr1], e0 = ssd_exp2(L0), e1 = ssd_exp2(L1);
#pragma unroll
      for (int nd = 0; nd < HALF / 8; ++nd) {
        acc[nd][0] *= e0; acc[nd][1] *= e0; acc[nd][2] *= e1; acc[nd][3] *= e1;
      }
      // the scores, weighted and masked, times x
#pragma unroll
      for (int kc = 0; kc < 4; ++kc) {
        if (kc > rb) continue;
        unsigned hi[4], lo[4];
#pragma unroll
        for (int q = 0; q < 2; ++q) {                // key tile q: a0, a2 the first eight tokens, a1, a3 the others
          const int nt = 2 * kc + q, s = nt * 8 + 2 * t;
          const float2 Ls = *reinterpret_cast<const float2*>(&cum[ih][s]), ds = *reinterpret_cast<const float2*>(&dts[ih][s]);
          float v0 = sc[nt][0] * (ssd_exp2(L0 - Ls.x) * ds.x), v1 = sc[nt][1] * (ssd_exp2(L0 - Ls.y) * ds.y);
          float v2 = sc[nt][2] * (ssd_exp2(L1 - Ls.x) * ds.x), v3 = sc[nt][3] * (ssd_exp2(L1 - Ls.y) * ds.y);
          if (kc == rb) {                            // the tile on the diagonal: nothing from later tokens
            v0 = s <= tr0 ? v0 : 0.0f; v1 = s < tr0 ? v1 : 0.0f;
            v2 = s <= tr1 ? v2 : 0.0f; v3 = s < tr1 ? v3 : 0.0f;
          }
          ssd_split2(v0, v1, hi[2 * q], lo[2 * q]);
          ssd_split2(v2, v3, hi[2 * q + 1], lo[2 * q + 1]);
        }
#pragma unroll
        for (int nd = 0; nd < HALF / 16; ++nd) {
          unsigned b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, Xs + (kc * 16 + (mi & 1) * 8 + l8) * XS + cb + nd * 16 + (mi >> 1) * 8);
          mma16816(acc[2 * nd], hi[0], hi[1], hi[2], hi[3], b0, b1);
          mma16816(acc[2 * nd + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
          mma16816(acc[2 * nd], lo[0], lo[1], lo[2], lo[3], b0, b1);
          mma16816(acc[2 * nd + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
        }
      }
      const float dskip = a.dskip != nullptr ? a.dskip[h] : 0.0f;
#pragma unroll
      for (int nd = 0; nd < HALF / 8; ++nd)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int tr = half ? tr1 : tr0, v = cb + nd * 8 + 2 * t;
          if (tr >= w.n || v >= w.cols) continue;
          const float y0 = fmaf(dskip, __bfloat162float(Xs[tr * XS + v]), acc[nd][2 * half]);
          const float y1 = fmaf(dskip, __bfloat162float(Xs[tr * XS + v + 1]), acc[nd][2 * half + 1]);
          float* p = a.out + (size_t)(w.tok0 + tr) * a.ldo + (size_t)h * a.dv + w.v0 + v;
          if (pair) *reinterpret_cast<float2*>(p) = make_float2(y0, y1);
          else {
            p[0] = y0;
            if (v + 1 < w.cols) p[1] = y1;
          }
        }
    }
    __syncthreads();                                 // this head's stage may be overwritten
    if (stages == 1 && ih + 1 < w.nh) stage(ih + 1);
  }
}

// Chunks that a step of n_tokens tokens in n_seqs sequences can have (rows of the scratch arrays); 0: these sizes go
// token by token.
extern "C" int hb_ssd_chunks(int n_tokens, int n_seqs, int N, int dv) {
  if (N > 256 || N < 1 || dv < 1) return 0;
  return n_tokens / SC_Q + n_seqs;
}

// chunk_state [hb_ssd_chunks(..)][heads][N][dv], chunk_decay [hb_ssd_chunks(..)][heads]: scratch.
extern "C" int hb_ssd_chunked_bf16(const void* xbc, int ld, int b_off, int c_off, const float* dt, int lddt, const float* logd,
                                   const float* dt_bias, const float* a_log, const float* dskip, float* state, const int* seq_slot,
                                   const int* seq_start, float* out, int ldo, int n_seqs, int max_q_len, int heads, int groups,
                                   int N, int dv, float* chunk_state, float* chunk_decay, void* stream) {
  SS_CHECKS("ssd_chunked");
  HB_REQUIRE(max_q_len > 0 && chunk_state != nullptr && chunk_decay != nullptr && ((uintptr_t)chunk_state & 15) == 0,
             "ssd_chunked: needs tokens and scratch (16-byte aligned)");
  HB_REQUIRE(N <= 256, "ssd_chunked: %d state rows per head exceed the supported maximum 256", N);
  HB_REQUIRE(((uintptr_t)out & 7) == 0, "ssd_chunked: the output must be 8-byte aligned");
  const int dvm = dv <= 32 ? 32 : dv <= 64 ? 64 : 128, vb = ceil_div(dv, dvm), chunks = ceil_div(max_q_len, SC_Q);
  const int vw = ceil_div(ceil_div(dv, vb), 16) * 16;      // the blocks of value channels are of one width, or nearly
  const SsdArgs a{xbc, ld, b_off, c_off, dt, lddt, logd, dt_bias, a_log, dskip, state, seq_slot, seq_start, out, ldo, heads, groups, N, dv,
                  0, chunk_state, chunk_decay, vw};
  const int vec = ld % 8 == 0 && b_off % 8 == 0 && c_off % 8 == 0 && N % 8 == 0 && dv % 8 == 0 && ((uintptr_t)xbc & 15) == 0;
  // heads of a group per CTA: as many as still leave every SM a CTA or two
  const int per = heads / groups;
  int hpc = per < SC_HEADS ? per : SC_HEADS;
  while (hpc > 1 && (long long)chunks * n_seqs * groups * ceil_div(per, hpc) * vb < 2LL * ssd_sms()) --hpc;
  const long long gy = (long long)groups * ceil_div(per, hpc) * vb;
  HB_REQUIRE(gy <= 65535, "ssd_chunked: too many heads or value channels");
  const int NP = (N + 15) / 16 * 16;
  const size_t row = (size_t)SC_Q * (NP + 8) * 2, xrow = (size_t)SC_Q * (dvm + 8) * 2, st = xrow + 2 * (size_t)NP * (dvm + 8) * 2;
  const size_t sm1 = row + 4 * xrow;
  // two CTAs an SM hide each other's loads; where only one fits, it fetches the next head's ahead
  const int stages = hpc > 1 && 2 * row + st > 110 * 1024 && 2 * row + 2 * st <= 220 * 1024 ? 2 : 1;
  const size_t sm3 = 2 * row + stages * st;
  const dim3 grid(chunks, (unsigned)gy, n_seqs);
  cudaStream_t s = (cudaStream_t)stream;
#define SC_GO(KERNEL, SM, ...)                                                                                     \
  do {                                                                                                             \
    cudaError_t e = cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(SM));          \
    if (e != cudaSuccess) HB_FAIL(3, "ssd_chunked: cannot reserve %d bytes of shared memory: %s", (int)(SM), cudaGetErrorString(e)); \
    hb_launch(KERNEL, grid, dim3(SC_T), SM, s, a, vb, vec, __VA_ARGS__);                                           \
  } while (0)
  if (dvm == 32) SC_GO(ssd_chunk_state_kernel<32>, sm1, hpc);
  else if (dvm == 64) SC_GO(ssd_chunk_state_kernel<64>, sm1, hpc);
  else SC_GO(ssd_chunk_state_kernel<128>, sm1, hpc);
  HB_CHECK_LAUNCH("ssd_chunk_state");
  if (dv % 8 == 0)
    hb_launch(ssd_state_pass_kernel<8>, dim3(ceil_div(N * dv / 8, 128), heads, n_seqs), dim3(128), 0, s, a);
  else
    hb_launch(ssd_state_pass_kernel<1>, dim3(ceil_div(N * dv, 128), heads, n_seqs), dim3(128), 0, s, a);
  HB_CHECK_LAUNCH("ssd_state_pass");
  if (dvm == 32) SC_GO(ssd_chunk_out_kernel<32>, sm3, hpc, stages);
  else if (dvm == 64) SC_GO(ssd_chunk_out_kernel<64>, sm3, hpc, stages);
  else SC_GO(ssd_chunk_out_kernel<128>, sm3, hpc, stages);
#undef SC_GO
  HB_CHECK_LAUNCH("ssd_chunk_out");
  return 0;
}
