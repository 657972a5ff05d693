// A residual stream of n copies ("hyper-connections"): a sublayer reads a mixture of the copies, its result joins
// them through a matrix.  x is [tokens][n][D] floats.  For a sublayer with result y and the next one's input weights:
//
//   x_t <- sum_s M[s][t] x_s + b_t y                 every copy from the old ones       (y null: x stays as it is)
//   u    = sum_t a_t x_t                             a null: the plain sum
//   h    = (u - mean u) / sqrt(mean (u - mean u)^2 + eps) * w (+ bias)                  (h null: not asked for)
//          or, as an RMS norm, u / sqrt(mean u^2 + eps) * w (+ bias)
//
// in one pass: between two sublayers every copy is read and written once.  A CTA per row; a thread holds the n values
// of its columns in registers, u lies in shared memory until its mean and variance are known.  All float; h leaves in
// the activation type.
#include "api.h"
#include "common.cuh"

#define ST_MAX_STREAMS 16

struct JoinArgs {
  float* x;
  const float* y; int ldy;       // null: no update
  const float* mix;              // [n][n], from, to
  const float* out_w;            // [n]
  const float* in_w;             // [n] or null
  const float* w; const float* bias; float eps; int rms;
  void* h;                       // null: only the update
  const int* rows;               // h row r comes from row rows[r] of x (null: r); only without an update
  int n, D;
};

template <typename T> __device__ __forceinline__ void st_store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void st_store4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void st_store4<bf16>(bf16* p, float a, float b, float c, float d) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 v;
  v.x = *reinterpret_cast<const unsigned*>(&lo);
  v.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = v;
}

// NS copies at compile time; V columns a thread takes at once (4 with 16-byte accesses, or 1).
template <typename T, int NS, int V>
__global__ void __launch_bounds__(512) streams_kernel(JoinArgs a) {
  extern __shared__ __align__(16) float u[];     // [D]
  __shared__ float red[32];
  __shared__ float mix[NS * NS], ow[NS], iw[NS];
  pdl_wait();
  pdl_launch();
  const int r = blockIdx.x, D = a.D;
  for (int i = threadIdx.x; i < NS * NS; i += blockDim.x) mix[i] = a.y ? a.mix[i] : 0.0f;
  for (int i = threadIdx.x; i < NS; i += blockDim.x) {
    ow[i] = a.y ? a.out_w[i] : 0.0f;
    iw[i] = a.in_w ? a.in_w[i] : 1.0f;
  }
  __syncthreads();
  float* x = a.x + (size_t)(a.rows ? a.rows[r] : r) * NS * D;
  const float* y = a.y ? a.y + (size_t)r * a.ldy : nullptr;
  float sum = 0.0f;
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V) {
    float v[NS][V];
#pragma unroll
    for (int s = 0; s < NS; ++s) {
      if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(x + (size_t)s * D + c);
        v[s][0] = f.x; v[s][1] = f.y; v[s][2] = f.z; v[s][3] = f.w;
      } else {
        v[s][0] = x[(size_t)s * D + c];
      }
    }
    if (y) {
      float yv[V];
      if constexpr (V == 4) {
        const float4 f = *reinterpret_cast<const float4*>(y + c);
        yv[0] = f.x; yv[1] = f.y; yv[2] = f.z; yv[3] = f.w;
      } else {
        yv[0] = y[c];
      }
      float nv[NS][V];
#pragma unroll
      for (int t = 0; t < NS; ++t)
#pragma unroll
        for (int j = 0; j < V; ++j) {
          float z = ow[t] * yv[j];
#pragma unroll
          for (int s = 0; s < NS; ++s) z = fmaf(mix[s * NS + t], v[s][j], z);
          nv[t][j] = z;
        }
#pragma unroll
      for (int t = 0; t < NS; ++t) {
        if constexpr (V == 4) *reinterpret_cast<float4*>(x + (size_t)t * D + c) = make_float4(nv[t][0], nv[t][1], nv[t][2], nv[t][3]);
        else x[(size_t)t * D + c] = nv[t][0];
#pragma unroll
        for (int j = 0; j < V; ++j) v[t][j] = nv[t][j];
      }
    }
    if (a.h) {
#pragma unroll
      for (int j = 0; j < V; ++j) {
        float z = 0.0f;
#pragma unroll
        for (int s = 0; s < NS; ++s) z = fmaf(iw[s], v[s][j], z);
        u[c + j] = z;
        sum += z;
      }
    }
  }
  if (a.h == nullptr) return;
  float mean = 0.0f;
  if (!a.rms) mean = block_sum(sum, red) / (float)D;
  float q = 0.0f;                     // a thread reads only what it wrote itself
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V)
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float d = u[c + j] - mean;
      q = fmaf(d, d, q);
    }
  const float inv = 1.0f / sqrtf(block_sum(q, red) / (float)D + a.eps);
  T* h = (T*)a.h + (size_t)r * D;
  for (int c = threadIdx.x * V; c < D; c += blockDim.x * V) {
    float o[V];
#pragma unroll
    for (int j = 0; j < V; ++j) o[j] = ((u[c + j] - mean) * inv) * a.w[c + j] + (a.bias ? a.bias[c + j] : 0.0f);
    if constexpr (V == 4) st_store4<T>(h + c, o[0], o[1], o[2], o[3]);
    else h[c] = from_f32<T>(o[0]);
  }
}

template <typename T, int NS>
static int streams_launch(const JoinArgs& a, int n_rows, bool vec, cudaStream_t s) {
  const size_t smem = a.h ? (size_t)a.D * sizeof(float) : 0;
  HB_REQUIRE(smem <= 200 * 1024, "streams_join: rows of %d numbers do not fit a block's shared memory", a.D);
  const int cols = vec && NS <= 6 ? a.D / 4 : a.D;
  const int threads = cols >= 512 ? 512 : cols >= 256 ? 256 : 128;
  if constexpr (NS <= 6) {      // more copies: their values would not fit a thread's registers four columns at a time
    if (vec) {
      if (smem > 48 * 1024) cudaFuncSetAttribute(streams_kernel<T, NS, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      hb_launch(streams_kernel<T, NS, 4>, dim3(n_rows), dim3(threads), smem, s, a);
      HB_CHECK_LAUNCH("streams_join");
      return 0;
    }
  }
  {
    if (smem > 48 * 1024) cudaFuncSetAttribute(streams_kernel<T, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    hb_launch(streams_kernel<T, NS, 1>, dim3(n_rows), dim3(threads), smem, s, a);
  }
  HB_CHECK_LAUNCH("streams_join");
  return 0;
}

extern "C" int hb_streams_join(int dtype, float* x, int n, const float* y, int ldy, const float* mix, const float* out_w,
                               const float* in_w, const float* w, const float* bias, float eps, int rms, void* h,
                               const int* rows, int n_rows, int D, void* stream) {
  HB_REQUIRE(n_rows > 0 && D > 0, "streams_join: sizes must be positive");
  HB_REQUIRE(n >= 1 && n <= ST_MAX_STREAMS, "streams_join: %d copies of the stream are outside the supported range 1..%d", n, ST_MAX_STREAMS);
  HB_REQUIRE(y == nullptr || (mix != nullptr && out_w != nullptr), "streams_join: a result needs the matrix and the output weights");
  HB_REQUIRE(y != nullptr || h != nullptr, "streams_join: nothing to do");
  HB_REQUIRE(h == nullptr || w != nullptr, "streams_join: the norm needs its weight");
  HB_REQUIRE(rows == nullptr || y == nullptr, "streams_join: rows are chosen only where nothing is updated");
  const uintptr_t ptrs = (uintptr_t)x | (uintptr_t)y | (uintptr_t)h;
  const bool vec = D % 4 == 0 && (y == nullptr || ldy % 4 == 0) && (ptrs & 15) == 0;
  const JoinArgs a{x, y, ldy, mix, out_w, in_w, w, bias, eps, rms, h, rows, n, D};
  cudaStream_t s = (cudaStream_t)stream;
#define ST_GO(NS) case NS: return dtype == HB_F32 ? streams_launch<float, NS>(a, n_rows, vec, s) : streams_launch<bf16, NS>(a, n_rows, vec, s)
  switch (n) {
    ST_GO(1); ST_GO(2); ST_GO(3); ST_GO(4); ST_GO(5); ST_GO(6); ST_GO(7); ST_GO(8);
    ST_GO(9); ST_GO(10); ST_GO(11); ST_GO(12); ST_GO(13); ST_GO(14); ST_GO(15); ST_GO(16);
  }
#undef ST_GO
  HB_FAIL(2, "streams_join: %d copies", n);
}
