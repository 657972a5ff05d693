// What lies between the q/k/v product and attention for a mixer that norms q and k over the whole projection,
// rotates pairs by angles taken from the position, and keeps its values rotated too:
//
//   q <- q / sqrt(mean(q^2) + eps) * wq         over all heads of the row at once, or over each head's channels with one
//                                               weight for all heads (likewise k; optional)
//   pair m of the first `rot` channels of every q and k head turns by  p * fqk[m]
//   pair m of all dv channels of every v head turns by                p * fv[m]      (optional)
//   v <- (1 - lambda) v + lambda v'              v': a row of values that another layer of the step left as floats (optional);
//                                               a layer can leave its own rows (with their bias) for others
//   cos and sin of q's and k's angles are multiplied by one constant (scaled frequencies); a bias vector may be added
//   to the row before anything else
//   (u, v) -> (u cos a - v sin a, v cos a + u sin a);  pair m is (2m, 2m + 1) ("interleaved") or (m, m + n/2) ("halves")
//
// With `maps` > 1 a head has that many queries and keys of dk channels (attention maps over one value): the query of
// map m becomes a query head of its own whose channels m dk .. (m + 1) dk are set and whose others are zero, a key head
// holds its maps side by side, so the score of query (h, m) with a key is the score of map m alone.
//
// The product's rows arrive as floats [q: nh x maps x dk | k: nkv x maps x dk | v: nkv x dv]; q leaves in the activation type with
// heads of `hd` channels, k and v go into the paged cache whose heads have `hd` channels as well.  hd >= max(maps dk, dv):
// channels beyond those are written as zeros, so an attention kernel over heads of hd sees the same scores and
// returns the values' channels followed by zeros.  Angles are float products of the integer position and a float
// frequency, sine and cosine are the accurate ones.
//
//   hb_rotate_heads_back    y[t, h, :dv] = a head's attention result turned by -p (pair m by -p * fv[m]), compacted
//                           from heads of hd channels to heads of dv
//   hb_head_gate            y[t, h, :dv] = a head's attention result times sigmoid(g[t, h]) (one number per token and
//                           head; g null: as it is), compacted likewise
#include "api.h"
#include "common.cuh"

struct RotPrepArgs {
  const float* rows; int ld;
  const float* bias;               // in the rows' layout, added first; null: none
  const float* wq; const float* wk; float eps; int norm;      // norm: 0 none, 1 over the whole projection, 2 per head
  const float* fqk; int rot; int halves; float mscale;
  const float* fv;                 // null: values are stored as they are
  const int* tok_seq; const int* tok_pos; const int* seq_pages; int pages_stride;
  void* q_out; int ldq;
  void* kcache; void* vcache;
  int nh, nkv, maps, dk, dv, hd, page_size, write_cache;
  const float* blend; float lambda;      // [tokens][nkv * dv]: v <- (1 - lambda) v + lambda blend; null: as they are
  float* keep;                           // [tokens][nkv * dv]: receives v (with its bias, before any blending); or null
};

// own * cos + (-/+ partner) * sin for channel j of a head whose first `rot` channels are rotated; cs holds the
// token's cosines of all pairs, then the sines
__device__ __forceinline__ float turn_channel(const float* head, const float* bias, const float* w, float inv, int j, int rot,
                                              int halves, const float* cs) {
  const float own = (head[j] + (bias ? bias[j] : 0.0f)) * inv * (w ? w[j] : 1.0f);
  if (j >= rot) return own;
  const int half = rot >> 1;
  int m, partner;
  bool first;
  if (halves) {
    first = j < half;
    m = first ? j : j - half;
    partner = first ? j + half : j - half;
  } else {
    first = (j & 1) == 0;
    m = j >> 1;
    partner = j ^ 1;
  }
  const float other = (head[partner] + (bias ? bias[partner] : 0.0f)) * inv * (w ? w[partner] : 1.0f);
  const float c = cs[m], s = cs[half + m];
  return first ? own * c - other * s : own * c + other * s;
}

// The same for channels j .. j + 3 of a head at once: every size involved is a multiple of 4 (with halves, the half too).
__device__ __forceinline__ float4 turn_channels4(const float* head, const float* bias, const float* w, float inv, int j, int rot,
                                                 int halves, const float* cs) {
  auto value = [&](int i) {
    float4 x = *reinterpret_cast<const float4*>(head + i);
    if (bias) {
      const float4 b = *reinterpret_cast<const float4*>(bias + i);
      x.x += b.x; x.y += b.y; x.z += b.z; x.w += b.w;
    }
    x.x *= inv; x.y *= inv; x.z *= inv; x.w *= inv;
    if (w) {
      const float4 k = *reinterpret_cast<const float4*>(w + i);
      x.x *= k.x; x.y *= k.y; x.z *= k.z; x.w *= k.w;
    }
    return x;
  };
  const float4 own = value(j);
  if (j >= rot) return own;
  const int half = rot >> 1;
  if (halves) {
    const bool first = j < half;
    const int m = first ? j : j - half;
    const float4 other = value(first ? j + half : m);
    const float4 c = *reinterpret_cast<const float4*>(cs + m);
    float4 s = *reinterpret_cast<const float4*>(cs + half + m);
    if (first) { s.x = -s.x; s.y = -s.y; s.z = -s.z; s.w = -s.w; }
    return make_float4(own.x * c.x + other.x * s.x, own.y * c.y + other.y * s.y, own.z * c.z + other.z * s.z, own.w * c.w + other.w * s.w);
  }
  const int m = j >> 1;
  const float2 c = *reinterpret_cast<const float2*>(cs + m), s = *reinterpret_cast<const float2*>(cs + half + m);
  return make_float4(own.x * c.x - own.y * s.x, own.y * c.x + own.x * s.x, own.z * c.y - own.w * s.y, own.w * c.y + own.z * s.y);
}
template <typename T> __device__ __forceinline__ void rot_store4(T* p, float4 v);
template <> __device__ __forceinline__ void rot_store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void rot_store4<bf16>(bf16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned*>(&lo);
  u.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = u;
}

// One warp: 1 / rms of a head's n numbers (plus a bias).
__device__ __forceinline__ float head_inv_rms(const float* head, const float* bias, int n, float eps) {
  float s = 0.0f;
  for (int i = threadIdx.x & 31; i < n; i += 32) {
    const float x = head[i] + (bias ? bias[i] : 0.0f);
    s = fmaf(x, x, s);
  }
  return 1.0f / sqrtf(warp_sum(s) / (float)n + eps);
}

// V4: four channels a lane (see turn_channels4).
template <typename T, bool V4>
__global__ void __launch_bounds__(256) qkv_rotary_cache_kernel(RotPrepArgs a) {
  extern __shared__ __align__(16) float tab[];          // cos and sin of the token's angles: [rot] for q and k, [dv] for values
  __shared__ float red[32];
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x, p = a.tok_pos[t];
  const float pos = (float)p;
  float* tab_v = tab + a.rot;
  for (int m = threadIdx.x; m < a.rot / 2; m += blockDim.x) {
    float s, c;
    sincosf(pos * a.fqk[m], &s, &c);
    tab[m] = c * a.mscale;
    tab[a.rot / 2 + m] = s * a.mscale;
  }
  if (a.fv)
    for (int m = threadIdx.x; m < a.dv / 2; m += blockDim.x) {
      float s, c;
      sincosf(pos * a.fv[m], &s, &c);
      tab_v[m] = c;
      tab_v[a.dv / 2 + m] = s;
    }
  __syncthreads();
  const int qn = a.nh * a.maps * a.dk, kn = a.nkv * a.maps * a.dk;
  const float* q = a.rows + (size_t)t * a.ld;
  const float* k = q + qn;
  const float* v = k + kn;
  const float* bq = a.bias;
  const float* bk = a.bias ? a.bias + qn : nullptr;
  const float* bv = a.bias ? a.bias + qn + kn : nullptr;
  float inv_q = 1.0f, inv_k = 1.0f;
  if (a.norm == 1) {
    float sq = 0.0f, sk = 0.0f;
    for (int i = threadIdx.x; i < qn; i += blockDim.x) {
      const float x = q[i] + (bq ? bq[i] : 0.0f);
      sq = fmaf(x, x, sq);
    }
    for (int i = threadIdx.x; i < kn; i += blockDim.x) {
      const float x = k[i] + (bk ? bk[i] : 0.0f);
      sk = fmaf(x, x, sk);
    }
    sq = block_sum(sq, red);
    sk = block_sum(sk, red);
    inv_q = 1.0f / sqrtf(sq / (float)qn + a.eps);
    inv_k = 1.0f / sqrtf(sk / (float)kn + a.eps);
  }
  // map m of a head lies in channels m * dk ..: a query of map m is zero elsewhere, a key holds all maps side by side
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
  for (int h = warp; h < a.nh * a.maps; h += nwarp) {      // a warp per head: nothing is divided channel by channel
    const size_t at = (size_t)h * a.dk;
    const float* hb = bq ? bq + at : nullptr;
    const float* hw = a.norm == 2 ? a.wq : a.wq ? a.wq + at : nullptr;
    if (a.norm == 2) inv_q = head_inv_rms(q + at, hb, a.dk, a.eps);
    const int off = (h % a.maps) * a.dk;
    T* qo = (T*)a.q_out + (size_t)t * a.ldq + (size_t)h * a.hd;
    if constexpr (V4) {
      for (int i = lane * 4; i < a.hd; i += 128) {
        const int j = i - off;
        float4 r = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (j >= 0 && j < a.dk) r = turn_channels4(q + at, hb, hw, inv_q, j, a.rot, a.halves, tab);
        rot_store4<T>(qo + i, r);
      }
      continue;
    }
#pragma unroll 4
    for (int i = lane; i < a.hd; i += 32) {
      const int j = i - off;
      float r = 0.0f;
      if (j >= 0 && j < a.dk) r = turn_channel(q + at, hb, hw, inv_q, j, a.rot, a.halves, tab);
      qo[i] = from_f32<T>(r);
    }
  }
  if (!a.write_cache) return;
  const int page = a.seq_pages[(size_t)a.tok_seq[t] * a.pages_stride + p / a.page_size];
  const size_t in_page = (size_t)(p % a.page_size);
  for (int u = warp; u < 2 * a.nkv; u += nwarp) {          // key heads and value heads
    const int g = u >> 1;
    const size_t at = (((size_t)page * a.nkv + g) * a.page_size + in_page) * a.hd;
    if (u & 1) {
      T* vo = (T*)a.vcache + at;
      const float* hv = v + (size_t)g * a.dv;
      const float* hb = bv ? bv + (size_t)g * a.dv : nullptr;
      const size_t vrow = ((size_t)t * a.nkv + g) * a.dv;
      if constexpr (V4) {
        for (int j = lane * 4; j < a.hd; j += 128) {
          float4 r = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
          if (j < a.dv) {
            r = turn_channels4(hv, hb, nullptr, 1.0f, j, a.fv ? a.dv : 0, a.halves, tab_v);
            if (a.keep) *reinterpret_cast<float4*>(a.keep + vrow + j) = r;
            if (a.blend) {
              const float4 f = *reinterpret_cast<const float4*>(a.blend + vrow + j);
              const float k = 1.0f - a.lambda;
              r = make_float4(k * r.x + a.lambda * f.x, k * r.y + a.lambda * f.y, k * r.z + a.lambda * f.z, k * r.w + a.lambda * f.w);
            }
          }
          rot_store4<T>(vo + j, r);
        }
        continue;
      }
#pragma unroll 4
      for (int j = lane; j < a.hd; j += 32) {
        float r = 0.0f;
        if (j < a.dv) {
          r = turn_channel(hv, hb, nullptr, 1.0f, j, a.fv ? a.dv : 0, a.halves, tab_v);
          if (a.keep) a.keep[vrow + j] = r;
          if (a.blend) r = (1.0f - a.lambda) * r + a.lambda * a.blend[vrow + j];
        }
        vo[j] = from_f32<T>(r);
      }
      continue;
    }
    T* ko = (T*)a.kcache + at;
    if (a.norm == 2) inv_k = head_inv_rms(k + (size_t)g * a.dk, bk ? bk + (size_t)g * a.dk : nullptr, a.dk, a.eps);
    int m = 0, first = 0;                                   // the map that channel j belongs to
    if constexpr (V4) {
      for (int j = lane * 4; j < a.hd; j += 128) {
        while (m < a.maps && j - first >= a.dk) { ++m; first += a.dk; }
        const size_t head = (size_t)(g * a.maps + m) * a.dk;
        float4 r = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (m < a.maps)
          r = turn_channels4(k + head, bk ? bk + head : nullptr, a.wk ? a.wk + (a.norm == 2 ? 0 : head) : nullptr, inv_k, j - first, a.rot, a.halves, tab);
        rot_store4<T>(ko + j, r);
      }
      continue;
    }
    for (int j = lane; j < a.hd; j += 32) {
      float r = 0.0f;
      while (m < a.maps && j - first >= a.dk) { ++m; first += a.dk; }
      const size_t head = (size_t)(g * a.maps + m) * a.dk;
      if (m < a.maps) r = turn_channel(k + head, bk ? bk + head : nullptr, a.wk ? a.wk + (a.norm == 2 ? 0 : head) : nullptr, inv_k, j - first, a.rot, a.halves, tab);
      ko[j] = from_f32<T>(r);
    }
  }
}

extern "C" int hb_qkv_rotary_cache(int dtype, const float* rows, int ld, const float* bias, const float* wq, const float* wk, float eps,
                                   int norm, const float* fqk, int rot, int halves, float mscale, const float* fv, const int* tok_seq,
                                   const int* tok_pos, const int* seq_pages, int pages_stride, void* q_out, int ldq, void* kcache,
                                   void* vcache, int n_tokens, int nh, int nkv, int maps, int dk, int dv, int hd, int page_size,
                                   int write_cache, const float* blend, float lambda, float* keep, void* stream) {
  HB_REQUIRE(n_tokens > 0 && nh > 0 && nkv > 0 && maps > 0 && dk > 0 && dv > 0 && page_size > 0, "qkv_rotary_cache: sizes must be positive");
  HB_REQUIRE(hd >= maps * dk && hd >= dv, "qkv_rotary_cache: cache heads of %d channels cannot hold keys of %d x %d and values of %d", hd, maps, dk, dv);
  HB_REQUIRE(rot >= 0 && rot <= dk && rot % 2 == 0, "qkv_rotary_cache: %d rotated channels must be even and at most %d", rot, dk);
  HB_REQUIRE(norm >= 0 && norm <= 2 && (norm == 0 || (wq != nullptr && wk != nullptr)), "qkv_rotary_cache: a norm needs both its weights");
  HB_REQUIRE(norm != 2 || maps == 1, "qkv_rotary_cache: a norm per head serves one map per head");
  HB_REQUIRE((blend == nullptr && keep == nullptr) || (fv == nullptr && write_cache), "qkv_rotary_cache: values that are blended or kept are stored and not rotated");
  HB_REQUIRE(rot == 0 || fqk != nullptr, "qkv_rotary_cache: rotated channels need their frequencies");
  HB_REQUIRE(fv == nullptr || dv % 2 == 0, "qkv_rotary_cache: rotated values need an even size, got %d", dv);
  // a step that stores nothing (it reads another layer's keys and values) brings rows of queries only
  HB_REQUIRE(ld >= nh * maps * dk + (write_cache ? nkv * (maps * dk + dv) : 0) && ldq >= nh * maps * hd, "qkv_rotary_cache: rows are shorter than their heads");
  const size_t smem = (size_t)(rot + (fv ? dv : 0)) * sizeof(float);
  HB_REQUIRE(smem <= 48 * 1024, "qkv_rotary_cache: %d rotated channels exceed a block's shared memory", rot);
  RotPrepArgs a{rows, ld, bias, wq, wk, eps, norm, fqk, rot, halves, mscale, fv, tok_seq, tok_pos, seq_pages, pages_stride, q_out, ldq,
                kcache, vcache, nh, nkv, maps, dk, dv, hd, page_size, write_cache, blend, lambda, keep};
  const uintptr_t in_ptrs = (uintptr_t)rows | (uintptr_t)bias | (uintptr_t)wq | (uintptr_t)wk | (uintptr_t)blend | (uintptr_t)keep;
  const uintptr_t out_ptrs = (uintptr_t)q_out | (uintptr_t)kcache | (uintptr_t)vcache;
  const bool v4 = ((dk | dv | hd | ld | ldq) & 3) == 0 && (in_ptrs & 15) == 0 && (out_ptrs & 15) == 0 && rot % (halves ? 8 : 4) == 0 &&
                  (fv == nullptr || dv % (halves ? 8 : 4) == 0);
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == HB_F32) {
    if (v4) hb_launch(qkv_rotary_cache_kernel<float, true>, dim3(n_tokens), dim3(256), smem, s, a);
    else hb_launch(qkv_rotary_cache_kernel<float, false>, dim3(n_tokens), dim3(256), smem, s, a);
  } else {
    if (v4) hb_launch(qkv_rotary_cache_kernel<bf16, true>, dim3(n_tokens), dim3(256), smem, s, a);
    else hb_launch(qkv_rotary_cache_kernel<bf16, false>, dim3(n_tokens), dim3(256), smem, s, a);
  }
  HB_CHECK_LAUNCH("qkv_rotary_cache");
  return 0;
}

// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
rotate_heads_back_kernel(const T* __restrict__ att, int ld, int hd, const float* __restrict__ fv, int halves,
                         const int* __restrict__ tok_pos, T* __restrict__ y, int ldy, int nh, int dv) {
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x;
  const float pos = (float)tok_pos[t];
  const T* ar = att + (size_t)t * ld;
  T* yr = y + (size_t)t * ldy;
  const int half = dv >> 1;
  for (int i = threadIdx.x; i < nh * half; i += blockDim.x) {
    const int h = i / half, m = i - h * half;
    const int j0 = halves ? m : 2 * m, j1 = halves ? m + half : 2 * m + 1;
    const float u = to_f32(ar[(size_t)h * hd + j0]), w = to_f32(ar[(size_t)h * hd + j1]);
    float s = 0.0f, c = 1.0f;
    if (fv) sincosf(pos * fv[m], &s, &c);
    // the turn by -a
    yr[(size_t)h * dv + j0] = from_f32<T>(u * c + w * s);
    yr[(size_t)h * dv + j1] = from_f32<T>(w * c - u * s);
  }
}

extern "C" int hb_rotate_heads_back(int dtype, const void* att, int ld, int hd, const float* fv, int halves, const int* tok_pos,
                                    void* y, int ldy, int n_tokens, int nh, int dv, void* stream) {
  HB_REQUIRE(n_tokens > 0 && nh > 0 && dv > 0 && hd >= dv, "rotate_heads_back: sizes must be positive and heads wide enough");
  HB_REQUIRE(dv % 2 == 0, "rotate_heads_back: values of %d channels have no pairs", dv);
  if (dtype == HB_F32)
    hb_launch(rotate_heads_back_kernel<float>, dim3(n_tokens), dim3(128), 0, (cudaStream_t)stream, (const float*)att, ld, hd, fv,
              halves, tok_pos, (float*)y, ldy, nh, dv);
  else
    hb_launch(rotate_heads_back_kernel<bf16>, dim3(n_tokens), dim3(128), 0, (cudaStream_t)stream, (const bf16*)att, ld, hd, fv,
              halves, tok_pos, (bf16*)y, ldy, nh, dv);
  HB_CHECK_LAUNCH("rotate_heads_back");
  return 0;
}

// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
head_gate_kernel(const T* __restrict__ att, int ld, int hd, const float* __restrict__ gate, int ldg, T* __restrict__ y, int ldy,
                 int nh, int dv) {
  pdl_wait();
  pdl_launch();
  const int t = blockIdx.x;
  const T* ar = att + (size_t)t * ld;
  T* yr = y + (size_t)t * ldy;
  for (int i = threadIdx.x; i < nh * dv; i += blockDim.x) {
    const int h = i / dv, j = i - h * dv;
    const float g = gate ? 1.0f / (1.0f + expf(-gate[(size_t)t * ldg + h])) : 1.0f;
    yr[i] = from_f32<T>(to_f32(ar[(size_t)h * hd + j]) * g);
  }
}

extern "C" int hb_head_gate(int dtype, const void* att, int ld, int hd, const float* gate, int ldg, void* y, int ldy,
                            int n_tokens, int nh, int dv, void* stream) {
  HB_REQUIRE(n_tokens > 0 && nh > 0 && dv > 0 && hd >= dv, "head_gate: sizes must be positive and heads wide enough");
  if (dtype == HB_F32)
    hb_launch(head_gate_kernel<float>, dim3(n_tokens), dim3(128), 0, (cudaStream_t)stream, (const float*)att, ld, hd, gate, ldg,
              (float*)y, ldy, nh, dv);
  else
    hb_launch(head_gate_kernel<bf16>, dim3(n_tokens), dim3(128), 0, (cudaStream_t)stream, (const bf16*)att, ld, hd, gate, ldg,
              (bf16*)y, ldy, nh, dv);
  HB_CHECK_LAUNCH("head_gate");
  return 0;
}


// ---------------------------------------------------------------------------------------------
// Two attention maps of a head over the same values, subtracted and normed:
//   o = a1 - lambda * a2;   y[t, h, :] = o / sqrt(mean(o^2) + eps) * factor       (over the dv value channels)
// att holds floats, the maps of head h at heads 2h and 2h + 1 of hd channels.  One warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(128)
difference_heads_kernel(const float* __restrict__ att, int ld, int hd, float lambda, float factor, float eps, T* __restrict__ y,
                        int ldy, int n_tokens, int nh, int dv) {
  pdl_wait();
  pdl_launch();
  const int lane = threadIdx.x & 31;
  const long long unit = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (unit >= (long long)n_tokens * nh) return;
  const int t = (int)(unit / nh), h = (int)(unit % nh);
  const float* a1 = att + (size_t)t * ld + (size_t)(2 * h) * hd;
  const float* a2 = a1 + hd;
  float ss = 0.0f;
  for (int i = lane; i < dv; i += 32) {
    const float o = a1[i] - lambda * a2[i];
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  const float k = factor / sqrtf(ss / (float)dv + eps);
  T* yr = y + (size_t)t * ldy + (size_t)h * dv;
  for (int i = lane; i < dv; i += 32) yr[i] = from_f32<T>((a1[i] - lambda * a2[i]) * k);
}

extern "C" int hb_difference_heads(int dtype, const float* att, int ld, int hd, float lambda, float factor, float eps, void* y,
                                   int ldy, int n_tokens, int nh, int dv, void* stream) {
  HB_REQUIRE(n_tokens > 0 && nh > 0 && dv > 0 && hd >= dv, "difference_heads: sizes must be positive and heads wide enough");
  const long long blocks = ceil_div_ll((long long)n_tokens * nh, 4);
  HB_REQUIRE(blocks < 2147483647LL, "difference_heads: too many (token, head) pairs");
  if (dtype == HB_F32)
    hb_launch(difference_heads_kernel<float>, dim3((unsigned)blocks), dim3(128), 0, (cudaStream_t)stream, att, ld, hd, lambda, factor,
              eps, (float*)y, ldy, n_tokens, nh, dv);
  else
    hb_launch(difference_heads_kernel<bf16>, dim3((unsigned)blocks), dim3(128), 0, (cudaStream_t)stream, att, ld, hd, lambda, factor,
              eps, (bf16*)y, ldy, n_tokens, nh, dv);
  HB_CHECK_LAUNCH("difference_heads");
  return 0;
}
