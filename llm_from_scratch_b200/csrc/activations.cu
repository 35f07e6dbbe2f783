// Element-wise activations of feed-forwards and heads: squared ReLU, and the scale and soft cap of logits.
#include "common.cuh"

namespace b200 {
namespace {

template <typename T, int E>
__global__ void __launch_bounds__(256) squared_relu_kernel(T* x, int64_t units) {
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < units;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    if constexpr (E > 1) {
      Pack p;
      p.u = reinterpret_cast<const uint4*>(x)[i];
#pragma unroll
      for (int k = 0; k < E; ++k) {
        const float r = fmaxf(to_float<T>(p.e[k]), 0.f);
        p.e[k] = from_float<T>(r * r);
      }
      reinterpret_cast<uint4*>(x)[i] = p.u;
    } else {
      const float r = fmaxf(to_float<T>(x[i]), 0.f);
      x[i] = from_float<T>(r * r);
    }
  }
}

__global__ void __launch_bounds__(256) softcap_kernel(float* z, int64_t n, float scale, float cap, float inv_cap) {
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const float v = z[i] * scale;
    z[i] = cap > 0.f ? cap * tanhf(v * inv_cap) : v;
  }
}

inline unsigned elementwise_grid(int64_t units) {
  const int64_t want = (units + 255) / 256;
  return static_cast<unsigned>(want < 148 * 32 ? want : 148 * 32);
}

}  // namespace
}  // namespace b200

extern "C" int b200_squared_relu(void* x, int64_t n, int32_t dtype, void* stream) {
  using namespace b200;
  if (n < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (n == 0) return B200_OK;
  if (!x) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = n % E == 0 && aligned16(x);
  const int64_t units = vec ? n / E : n;
  const unsigned grid = elementwise_grid(units);
  if (dtype == B200_DTYPE_F32) {
    if (vec) squared_relu_kernel<float, 4><<<grid, 256, 0, s>>>(static_cast<float*>(x), units);
    else squared_relu_kernel<float, 1><<<grid, 256, 0, s>>>(static_cast<float*>(x), units);
  } else {
    if (vec) squared_relu_kernel<__nv_bfloat16, 8><<<grid, 256, 0, s>>>(static_cast<__nv_bfloat16*>(x), units);
    else squared_relu_kernel<__nv_bfloat16, 1><<<grid, 256, 0, s>>>(static_cast<__nv_bfloat16*>(x), units);
  }
  return launch_result();
}

extern "C" int b200_softcap_logits(float* logits, int64_t n, float scale, float cap, void* stream) {
  using namespace b200;
  if (n < 0) return B200_ERR_ARG;
  if (n == 0) return B200_OK;
  if (!logits) return B200_ERR_ARG;
  softcap_kernel<<<elementwise_grid(n), 256, 0, static_cast<cudaStream_t>(stream)>>>(logits, n, scale, cap,
                                                                                    cap > 0.f ? 1.f / cap : 0.f);
  return launch_result();
}
