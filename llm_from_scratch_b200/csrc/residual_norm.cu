// fp32 residual of a decoder whose layers norm the sublayer's OUTPUT, one launch per sublayer boundary:
//
//   x <- x + y / sqrt(mean(y^2) + eps) * w        y: the sublayer's result, activation dtype
//   h  = x, rounded to the activation dtype       what the next sublayer reads, or with a final norm
//   h  = x / sqrt(mean(x^2) + eps) * final_w
//
// The first boundary starts x from the embedding row instead.  One CTA per token row; with the row in registers every
// load precedes the first reduction.
#include "common.cuh"

namespace b200 {
namespace {

struct ResArgs {
  float* x;                  // [T, d]
  const int64_t* tokens;     // [T] with embed, else null
  const void* embed;         // [vocab, d]
  int64_t vocab;
  const void* y;             // [T, d]
  const float* w;            // [d]
  const float* final_w;      // [d] or null
  float eps;
  void* h;                   // [T, d]
  int d;
  int32_t* status;
};

__device__ __forceinline__ float cta_sum(float v, float* scratch) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? scratch[lane] : 0.f);
}

template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  if constexpr (sizeof(T) == 2) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&a.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
  } else {
    return *reinterpret_cast<const float4*>(p);
  }
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 v) {
  if constexpr (sizeof(T) == 2)
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  else
    *reinterpret_cast<float4*>(p) = v;
}
__device__ __forceinline__ float sumsq(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

__device__ __forceinline__ int64_t embed_row(const ResArgs& a, int64_t row) {
  const int64_t tok = a.tokens[row];
  if (tok >= 0 && tok < a.vocab) return tok;
  if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
  return 0;
}

// N groups of four channels per thread, d a multiple of four
template <typename T, int N>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const ResArgs a) {
  __shared__ float scratch[2][32];
  const int d = a.d, step = blockDim.x * 4, first = threadIdx.x * 4;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * d;
  T* hr = static_cast<T*>(a.h) + row * d;
  float4 x[N], y[N], w[N], fw[N];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const T* src = a.embed ? static_cast<const T*>(a.embed) + embed_row(a, row) * d : static_cast<const T*>(a.y) + row * d;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = first + i * step;
    const bool in = c < d;
    y[i] = in ? load4<T>(src + c) : zero;
    x[i] = in && a.embed == nullptr ? *reinterpret_cast<const float4*>(xr + c) : zero;
    w[i] = in && a.embed == nullptr ? *reinterpret_cast<const float4*>(a.w + c) : zero;
    fw[i] = in && a.final_w ? *reinterpret_cast<const float4*>(a.final_w + c) : zero;
  }
  if (a.embed != nullptr) {
#pragma unroll
    for (int i = 0; i < N; ++i) x[i] = y[i];
  } else {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) ss += sumsq(y[i]);
    const float inv = rsqrtf(cta_sum(ss, scratch[0]) / static_cast<float>(d) + a.eps);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      x[i].x += y[i].x * inv * w[i].x;
      x[i].y += y[i].y * inv * w[i].y;
      x[i].z += y[i].z * inv * w[i].z;
      x[i].w += y[i].w * inv * w[i].w;
    }
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = first + i * step;
    if (c < d) *reinterpret_cast<float4*>(xr + c) = x[i];
  }
  if (a.final_w != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) ss += sumsq(x[i]);
    const float inv = rsqrtf(cta_sum(ss, scratch[1]) / static_cast<float>(d) + a.eps);
#pragma unroll
    for (int i = 0; i < N; ++i)
      x[i] = make_float4(x[i].x * inv * fw[i].x, x[i].y * inv * fw[i].y, x[i].z * inv * fw[i].z, x[i].w * inv * fw[i].w);
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = first + i * step;
    if (c < d) store4<T>(hr + c, x[i]);
  }
}

// any width
template <typename T>
__global__ void __launch_bounds__(256) residual_norm_any_kernel(const ResArgs a) {
  __shared__ float scratch[2][32];
  const int d = a.d;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * d;
  T* hr = static_cast<T*>(a.h) + row * d;
  const T* src = a.embed ? static_cast<const T*>(a.embed) + embed_row(a, row) * d : static_cast<const T*>(a.y) + row * d;
  float inv = 1.f;
  if (a.embed == nullptr) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) ss += to_float<T>(src[c]) * to_float<T>(src[c]);
    inv = rsqrtf(cta_sum(ss, scratch[0]) / static_cast<float>(d) + a.eps);
  }
  float ss = 0.f;
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    const float v = to_float<T>(src[c]);
    const float x = a.embed ? v : xr[c] + v * inv * a.w[c];
    xr[c] = x;
    ss += x * x;
    if (a.final_w == nullptr) hr[c] = from_float<T>(x);
  }
  if (a.final_w != nullptr) {
    inv = rsqrtf(cta_sum(ss, scratch[1]) / static_cast<float>(d) + a.eps);
    for (int c = threadIdx.x; c < d; c += blockDim.x) hr[c] = from_float<T>(xr[c] * inv * a.final_w[c]);
  }
}

template <typename T>
void launch(const ResArgs& a, int64_t rows, bool vec, cudaStream_t s) {
  const unsigned grid = static_cast<unsigned>(rows);
  const int groups = a.d / 4;
  if (vec && groups <= 1024) residual_norm_kernel<T, 1><<<grid, (groups + 31) / 32 * 32, 0, s>>>(a);
  else if (vec && groups <= 2048) residual_norm_kernel<T, 2><<<grid, (groups + 63) / 64 * 32, 0, s>>>(a);
  else residual_norm_any_kernel<T><<<grid, 256, 0, s>>>(a);
}

}  // namespace
}  // namespace b200

extern "C" int b200_residual_norm(float* x, const int64_t* tokens, const void* embed, int64_t vocab, const void* y,
                                  const float* norm_w, const float* final_w, float eps, void* h, int64_t rows, int32_t d,
                                  int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (rows < 0 || d <= 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!x || !h || (embed ? !tokens : (!y || !norm_w))) return B200_ERR_ARG;
  if (rows > 2147483647) return B200_ERR_TOO_LARGE;
  ResArgs a{x, tokens, embed, vocab, y, norm_w, final_w, eps, h, d, status};
  const bool vec = d % 4 == 0 && aligned16(x) && aligned16(h) && aligned16(embed ? embed : y) &&
                   (embed || aligned16(norm_w)) && (!final_w || aligned16(final_w));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) launch<float>(a, rows, vec, s);
  else launch<__nv_bfloat16>(a, rows, vec, s);
  return launch_result();
}
