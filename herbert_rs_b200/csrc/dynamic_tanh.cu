// A norm without statistics, N(x) = tanh(alpha * x) * w + b (alpha one number, w and b one per channel), alone and in the
// kernel that joins a block's result to the residual stream:
//
//   x[r, :] += mult * (y[r, :] + yb)              (float; yb: a bias of the result, or none; y null: x stays as it is)
//   h1[r, :] = N1(x[r, :]),  h2[r, :] = N2(x[r, :])   (activation type; either may be left out)
//
// Nothing here looks at more than one channel, so the stream is read and written once and both norms that the next block
// (or two sublayers side by side) begins with leave the same pass.  All arithmetic is float.
#include "api.h"
#include "common.cuh"

struct TanhNorm {
  float alpha;
  const float* w;
  const float* b;
  void* out;           // null: not asked for
};

// tanh in float; where the result is rounded to bfloat16 next, as 1 - 2 / (1 + e^{2z}) with the fast exponential and
// division (absolute error about 1e-7; e^{2z} = inf gives 1, 0 gives -1).
template <typename T> __device__ __forceinline__ float tanh_of(float z) {
  if constexpr (sizeof(T) == 4) return tanhf(z);
  else return 1.0f - __fdividef(2.0f, 1.0f + __expf(2.0f * z));
}

// V: channels per thread (4: every pointer on 16 bytes and every row length a multiple of 4).
template <typename T, int V>
__global__ void __launch_bounds__(256)
residual_tanh_kernel(const float* __restrict__ y, int ldy, const float* __restrict__ yb, float mult, float* x, const int* __restrict__ rows,
                     TanhNorm n1, TanhNorm n2, int dim, long long total) {
  pdl_wait();
  pdl_launch();
  const long long at = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (at >= total) return;
  const int r = (int)(at / dim), c = (int)(at - (long long)r * dim);
  float* xr = x + (size_t)(rows ? rows[r] : r) * dim + c;
  auto load = [](float* v, const float* p) {
    if constexpr (V == 4) {
      const float4 f = *reinterpret_cast<const float4*>(p);
      v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    } else v[0] = p[0];
  };
  float v[V];
  load(v, xr);
  if (y != nullptr) {
    float s[V];
    load(s, y + (size_t)r * ldy + c);
    if (yb != nullptr) {
      float bias[V];
      load(bias, yb + c);
#pragma unroll
      for (int j = 0; j < V; ++j) s[j] += bias[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = fmaf(mult, s[j], v[j]);
    if constexpr (V == 4) *reinterpret_cast<float4*>(xr) = make_float4(v[0], v[1], v[2], v[3]);
    else xr[0] = v[0];
  }
  auto norm = [&](const TanhNorm& n) {
    if (n.out == nullptr) return;
    float w[V], b[V], o[V];
    load(w, n.w + c);
    load(b, n.b + c);
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = fmaf(tanh_of<T>(n.alpha * v[j]), w[j], b[j]);
    T* p = (T*)n.out + (size_t)r * dim + c;
    if constexpr (V == 4 && sizeof(T) == 2) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(o[0], o[1]), hi = __floats2bfloat162_rn(o[2], o[3]);
      uint2 u;
      u.x = *reinterpret_cast<const unsigned*>(&lo);
      u.y = *reinterpret_cast<const unsigned*>(&hi);
      *reinterpret_cast<uint2*>(p) = u;
    } else if constexpr (V == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
    } else p[0] = from_f32<T>(o[0]);
  };
  norm(n1);
  norm(n2);
}

// rows (only without y): which rows of x the norms read, n_rows of them.
extern "C" int hb_residual_tanh(int dtype, const float* y, int ldy, const float* yb, float mult, float* x, const int* rows,
                                float alpha1, const float* w1, const float* b1, void* h1, float alpha2, const float* w2,
                                const float* b2, void* h2, int n_rows, int dim, void* stream) {
  HB_REQUIRE(n_rows > 0 && dim > 0 && (y == nullptr || ldy >= dim), "residual_tanh: sizes must be positive and rows at least dim apart");
  HB_REQUIRE(y == nullptr || rows == nullptr, "residual_tanh: a result joins every row of the stream, not chosen ones");
  HB_REQUIRE((h1 == nullptr || (w1 != nullptr && b1 != nullptr)) && (h2 == nullptr || (w2 != nullptr && b2 != nullptr)),
             "residual_tanh: a norm needs its weight and its bias");
  HB_REQUIRE(y != nullptr || h1 != nullptr || h2 != nullptr, "residual_tanh: nothing to do");
  const long long total = (long long)n_rows * dim;
  const uintptr_t ptrs = (uintptr_t)y | (uintptr_t)yb | (uintptr_t)x | (uintptr_t)w1 | (uintptr_t)b1 | (uintptr_t)h1 |
                         (uintptr_t)w2 | (uintptr_t)b2 | (uintptr_t)h2;
  const bool v4 = dim % 4 == 0 && (y == nullptr || ldy % 4 == 0) && (ptrs & 15) == 0;
  const long long blocks = ceil_div_ll(v4 ? total / 4 : total, 256);
  HB_REQUIRE(blocks < 2147483647LL, "residual_tanh: too many elements");
  const TanhNorm n1{alpha1, w1, b1, h1}, n2{alpha2, w2, b2, h2};
  cudaStream_t s = (cudaStream_t)stream;
  const dim3 grid((unsigned)blocks);
#define RT_GO(T, V) hb_launch(residual_tanh_kernel<T, V>, grid, dim3(256), 0, s, y, ldy, yb, mult, x, rows, n1, n2, dim, total)
  if (dtype == HB_F32) {
    if (v4) RT_GO(float, 4); else RT_GO(float, 1);
  } else {
    if (v4) RT_GO(bf16, 4); else RT_GO(bf16, 1);
  }
#undef RT_GO
  HB_CHECK_LAUNCH("residual_tanh");
  return 0;
}
