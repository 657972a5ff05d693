// What lies between the projection of a matrix-memory mixer (mLSTM) and its recurrence.  Per token and head, with the raw
// gates zi, zf from the projection and a cap c:
//
//   i = c tanh((zi + bi) / c)                       log of the input gate
//   f = log sigmoid(c tanh((zf + bf) / c))          log of the forget gate
//   m_t = max(f + m_(t-1), i)                       a running maximum; m before the first token is 0
//   S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T,     n_t likewise with k alone
//   o_t = s S_t^T q / (max(|s n_t . q|, e^(-m_t)) + eps)         s: the queries' scale
//
// The memory S and the vector n are one matrix here: the values get a column of ones behind them, so n is that column
// of the state, n . q the same column of the read-out, and the recurrence is the state-space kernels' (state_space.cu:
// a decay and a weight per token and head, which this file makes).  The division is the first thing the norm behind the
// recurrence does (linear_scan.cu, hb_gated_rmsnorm).
//
// The running maximum of a sequence is a float per head in its slot; a step continues from it.  The maximum over a
// step's tokens is taken as a scan (pairs (sum of f, best i after its decay) compose), so two cuttings of a prompt
// agree to float rounding.
#include "api.h"
#include "common.cuh"

#define MM_THREADS 256

struct MemPrepArgs {
  const float* rows; int ld;                 // the projection's float rows
  int q_off, k_off, v_off, i_off, f_off;
  const float* i_bias; const float* f_bias;  // [H]
  float cap;
  float* m_state;                            // [slots][H]
  const int* seq_slot; const int* seq_start;
  void* packed; int ldp;                     // [T][ldp]: values [H][dvp] (dv, a one, zeros), then keys [H][dk], then queries [H][dk]
  float* logd; float* weight; float* floor_;  // [T][H] each
  int n_tokens, n_seqs, H, dk, dv, dvp;
};

struct MaxPlus { float a, b; };              // m -> max(m + a, b)
__device__ __forceinline__ MaxPlus mp_then(MaxPlus x, MaxPlus y) { return {x.a + y.a, fmaxf(x.b + y.a, y.b)}; }

// One sequence and head: THREADS tokens at a time.  LOCAL: the unit is one warp; else the whole block.
template <bool LOCAL>
__device__ __forceinline__ void mem_gates(const MemPrepArgs& a, int b, int h, MaxPlus* parts) {
  constexpr int N = LOCAL ? 32 : MM_THREADS;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, i0 = LOCAL ? lane : (int)threadIdx.x;
  const int t0 = a.seq_start[b], t1 = a.seq_start[b + 1];
  float* ms = a.m_state + (size_t)a.seq_slot[b] * a.H + h;
  const float bi = a.i_bias[h], bf = a.f_bias[h], inv_cap = 1.0f / a.cap;
  float m_in = *ms;
  for (int c0 = t0; c0 < t1; c0 += N) {
    const int t = c0 + i0;
    const bool live = t < t1;
    float gi = 0.0f, gf = 0.0f;
    if (live) {
      const float* row = a.rows + (size_t)t * a.ld;
      gi = a.cap * tanhf((row[a.i_off + h] + bi) * inv_cap);
      const float z = a.cap * tanhf((row[a.f_off + h] + bf) * inv_cap);
      gf = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
    }
    MaxPlus p = live ? MaxPlus{gf, gi} : MaxPlus{0.0f, -INFINITY};      // past the end: nothing changes
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const MaxPlus q{__shfl_up_sync(0xffffffffu, p.a, o), __shfl_up_sync(0xffffffffu, p.b, o)};
      if (lane >= o) p = mp_then(q, p);
    }
    MaxPlus all;
    if constexpr (LOCAL) {
      all = {__shfl_sync(0xffffffffu, p.a, 31), __shfl_sync(0xffffffffu, p.b, 31)};
    } else {
      __syncthreads();                       // the parts of the chunk before have been read
      if (lane == 31) parts[warp] = p;
      __syncthreads();
      MaxPlus before{0.0f, -INFINITY};
      all = before;
      for (int w = 0; w < N / 32; ++w) {
        if (w == warp) before = all;
        all = mp_then(all, parts[w]);
      }
      p = mp_then(before, p);
    }
    const float m = fmaxf(m_in + p.a, p.b);
    float m_prev = __shfl_up_sync(0xffffffffu, m, 1);
    if (lane == 0) {
      m_prev = m_in;
      if (!LOCAL && warp > 0) {              // the maximum after the warps before this one
        MaxPlus q{0.0f, -INFINITY};
        for (int w = 0; w < warp; ++w) q = mp_then(q, parts[w]);
        m_prev = fmaxf(m_in + q.a, q.b);
      }
    }
    if (live) {
      const size_t o = (size_t)t * a.H + h;
      a.logd[o] = fminf(gf + m_prev - m, 0.0f);
      a.weight[o] = expf(gi - m);
      a.floor_[o] = expf(-m);
    }
    m_in = fmaxf(m_in + all.a, all.b);
  }
  if (i0 == 0 && t1 > t0) *ms = m_in;        // every thread read it before its first token
}

// Blocks 0 .. gate_blocks - 1: the gates; the others: one token's row each, rounded once and packed.
template <typename T, bool LOCAL>
__global__ void __launch_bounds__(MM_THREADS) mem_prepare_kernel(MemPrepArgs a, int gate_blocks, int v4) {
  __shared__ MaxPlus parts[MM_THREADS / 32];
  pdl_wait();
  pdl_launch();
  if ((int)blockIdx.x < gate_blocks) {
    const int u = LOCAL ? blockIdx.x * (MM_THREADS / 32) + (threadIdx.x >> 5) : blockIdx.x;
    if (u >= a.n_seqs * a.H) return;         // a whole warp, or nobody
    mem_gates<LOCAL>(a, u / a.H, u % a.H, parts);
    return;
  }
  const int t = blockIdx.x - gate_blocks;
  const float* row = a.rows + (size_t)t * a.ld;
  T* out = (T*)a.packed + (size_t)t * a.ldp;
  const int xn = a.H * a.dvp, kn = a.H * a.dk;
  if (v4) {
    auto put = [&](T* p, float4 f) {
      if constexpr (sizeof(T) == 4) {
        *reinterpret_cast<float4*>(p) = f;
      } else {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(f.x, f.y), hi = __floats2bfloat162_rn(f.z, f.w);
        uint2 u;
        u.x = *reinterpret_cast<const unsigned*>(&lo);
        u.y = *reinterpret_cast<const unsigned*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
      }
    };
    for (int c = threadIdx.x * 4; c < xn; c += MM_THREADS * 4) {
      const int h = c / a.dvp, j = c - h * a.dvp;
      float4 f = make_float4(j == a.dv ? 1.0f : 0.0f, 0.0f, 0.0f, 0.0f);
      if (j < a.dv) f = *reinterpret_cast<const float4*>(row + a.v_off + h * a.dv + j);
      put(out + c, f);
    }
    for (int c = threadIdx.x * 4; c < kn; c += MM_THREADS * 4) {
      put(out + xn + c, *reinterpret_cast<const float4*>(row + a.k_off + c));
      put(out + xn + kn + c, *reinterpret_cast<const float4*>(row + a.q_off + c));
    }
    return;
  }
  for (int c = threadIdx.x; c < xn; c += MM_THREADS) {
    const int h = c / a.dvp, j = c - h * a.dvp;
    out[c] = from_f32<T>(j < a.dv ? row[a.v_off + h * a.dv + j] : j == a.dv ? 1.0f : 0.0f);
  }
  for (int c = threadIdx.x; c < kn; c += MM_THREADS) {
    out[xn + c] = from_f32<T>(row[a.k_off + c]);
    out[xn + kn + c] = from_f32<T>(row[a.q_off + c]);
  }
}

extern "C" int hb_matrix_memory_prepare(int dtype, const float* rows, int ld, int q_off, int k_off, int v_off, int i_off, int f_off,
                                        const float* i_bias, const float* f_bias, float cap, float* m_state, const int* seq_slot,
                                        const int* seq_start, void* packed, int ldp, float* logd, float* weight, float* floor_,
                                        int n_tokens, int n_seqs, int max_q_len, int heads, int dk, int dv, int dvp, void* stream) {
  HB_REQUIRE(n_tokens > 0 && n_seqs > 0 && max_q_len > 0 && heads > 0 && dk > 0 && dv > 0, "matrix_memory_prepare: sizes must be positive");
  HB_REQUIRE(dvp > dv && ldp >= heads * (dvp + 2 * dk), "matrix_memory_prepare: heads of %d columns have no room for %d values and a one, or rows of %d are too short", dvp, dv, ldp);
  HB_REQUIRE(cap > 0.0f, "matrix_memory_prepare: the gates' cap must be > 0");
  const bool local = max_q_len <= 32;
  const long long units = (long long)n_seqs * heads, gate_blocks = local ? ceil_div_ll(units, MM_THREADS / 32) : units;
  HB_REQUIRE(gate_blocks + n_tokens < 2147483647LL, "matrix_memory_prepare: too many tokens or heads");
  const int v4 = ((dv | dvp | ld | ldp | q_off | k_off | v_off) & 3) == 0 && ((heads * dk) & 3) == 0 &&
                 (((uintptr_t)rows | (uintptr_t)packed) & 15) == 0;
  const MemPrepArgs a{rows, ld, q_off, k_off, v_off, i_off, f_off, i_bias, f_bias, cap, m_state, seq_slot, seq_start, packed, ldp,
                      logd, weight, floor_, n_tokens, n_seqs, heads, dk, dv, dvp};
  const dim3 grid((unsigned)(gate_blocks + n_tokens));
  cudaStream_t s = (cudaStream_t)stream;
#define MM_GO(T, LOCAL) hb_launch(mem_prepare_kernel<T, LOCAL>, grid, dim3(MM_THREADS), 0, s, a, (int)gate_blocks, v4)
  if (dtype == HB_F32) {
    if (local) MM_GO(float, true); else MM_GO(float, false);
  } else {
    if (local) MM_GO(bf16, true); else MM_GO(bf16, false);
  }
#undef MM_GO
  HB_CHECK_LAUNCH("matrix_memory_prepare");
  return 0;
}
