// Activations of feed-forwards and heads: squared ReLU, the polynomial of normed powers, a tanh GELU that scales rows of a
// token table, and the scale and soft cap of logits.
#include "sequences.cuh"

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

__device__ __forceinline__ float3 cta_sum3(float3 v, float3* scratch) {
  v = make_float3(warp_sum(v.x), warp_sum(v.y), warp_sum(v.z));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  v = lane < nw ? scratch[lane] : make_float3(0.f, 0.f, 0.f);
  return make_float3(warp_sum(v.x), warp_sum(v.y), warp_sum(v.z));
}

// out = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 per row, N(u) = u / sqrt(mean(u^2) + eps).  The three means come from one pass
// over the row; N accesses of E elements per thread stay in registers (N == 0: a second pass over memory).  A CTA per row.
template <typename T, int E, int N>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* z, int64_t stride, const float* coef, float eps, T* out, int W) {
  __shared__ float3 scratch[16];
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  z += blockIdx.x * stride;
  out += static_cast<int64_t>(blockIdx.x) * W;
  constexpr int KEEP = N > 0 ? N : 1;
  Pack keep[KEEP];
  const int step = blockDim.x * E, first = threadIdx.x * E;
  float3 ss = make_float3(0.f, 0.f, 0.f);
  auto add = [&](float v) {
    const float q = v * v;
    ss.x += q;
    ss.y += q * q;
    ss.z += q * q * q;
  };
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + i * step;
      keep[i].u = c < W ? *reinterpret_cast<const uint4*>(z + c) : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
#pragma unroll
      for (int e = 0; e < E; ++e) add(to_float<T>(keep[i].e[e]));
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) add(to_float<T>(z[c]));
  }
  ss = cta_sum3(ss, scratch);
  const float n = 1.f / static_cast<float>(W);
  const float a = coef[0] * rsqrtf(ss.x * n + eps), b = coef[1] * rsqrtf(ss.y * n + eps), c3 = coef[2] * rsqrtf(ss.z * n + eps);
  const float c0 = coef[3];
  auto value = [&](float v) { return ((c3 * v + b) * v + a) * v + c0; };
  if constexpr (N > 0) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + i * step;
      if (c >= W) continue;
#pragma unroll
      for (int e = 0; e < E; ++e) keep[i].e[e] = from_float<T>(value(to_float<T>(keep[i].e[e])));
      *reinterpret_cast<uint4*>(out + c) = keep[i].u;
    }
  } else {
    for (int c = threadIdx.x; c < W; c += blockDim.x) out[c] = from_float<T>(value(to_float<T>(z[c])));
  }
}

template <typename T>
void poly_norm(const void* z, int64_t stride, const float* coef, float eps, void* out, int64_t rows, int W, bool vec, cudaStream_t s) {
  constexpr int E = 16 / sizeof(T);
  const unsigned grid = static_cast<unsigned>(rows);
  const T* zp = static_cast<const T*>(z);
  T* op = static_cast<T*>(out);
  const int units = (W + E - 1) / E;
  auto threads = [&](int per) { return ((units + per - 1) / per + 31) / 32 * 32; };
  if (vec && units <= 512) poly_norm_kernel<T, E, 1><<<grid, threads(1), 0, s>>>(zp, stride, coef, eps, op, W);
  else if (vec && units <= 1024) poly_norm_kernel<T, E, 2><<<grid, threads(2), 0, s>>>(zp, stride, coef, eps, op, W);
  else if (vec && units <= 2048) poly_norm_kernel<T, E, 4><<<grid, threads(4), 0, s>>>(zp, stride, coef, eps, op, W);
  else if (vec && units <= 4096) poly_norm_kernel<T, E, 8><<<grid, 512, 0, s>>>(zp, stride, coef, eps, op, W);
  else poly_norm_kernel<T, E, 0><<<grid, 512, 0, s>>>(zp, stride, coef, eps, op, W);
}

// out[t] = gelu_tanh(u[t]) * table[tokens[t], first .. first + W - 1]; E elements per access.
// gelu_tanh(z) = z sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
template <typename T, int E>
__global__ void __launch_bounds__(256) gelu_table_kernel(const T* u, const T* table, int64_t table_width, int64_t vocab, int first,
                                                         const int64_t* tokens, T* out, int64_t rows, int W, int32_t* status) {
  const int units = W / E;
  const int64_t total = rows * units;
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t t = i / units;
    const int c = static_cast<int>(i - t * units) * E;
    int64_t tok = tokens[t];
    if (tok < 0 || tok >= vocab) {
      report(status, B200_ERR_BOUNDS);
      tok = 0;
    }
    const T* up = u + t * W + c;
    const T* tp = table + tok * table_width + first + c;
    Pack z, e;
    if constexpr (E > 1) {
      z.u = *reinterpret_cast<const uint4*>(up);
      e.u = *reinterpret_cast<const uint4*>(tp);
    } else {
      z.e[0] = up[0];
      e.e[0] = tp[0];
    }
#pragma unroll
    for (int k = 0; k < E; ++k) {
      const float v = to_float<T>(z.e[k]);
      z.e[k] = from_float<T>(v * sigmoid_for<T>(1.5957691216057308f * (v + 0.044715f * v * v * v)) * to_float<T>(e.e[k]));
    }
    if constexpr (E > 1) *reinterpret_cast<uint4*>(out + t * W + c) = z.u;
    else out[t * W + c] = z.e[0];
  }
}

template <typename T>
void gelu_table(const void* u, const void* table, int64_t table_width, int64_t vocab, int first, const int64_t* tokens, void* out,
                int64_t rows, int W, int32_t* status, cudaStream_t s) {
  constexpr int E = 16 / sizeof(T);
  const bool vec = W % E == 0 && table_width % E == 0 && first % E == 0 && aligned16(u) && aligned16(table) && aligned16(out);
  const int64_t blocks = (rows * (W / (vec ? E : 1)) + 255) / 256;
  const unsigned grid = static_cast<unsigned>(blocks < 148 * 32 ? blocks : 148 * 32);
  const T* up = static_cast<const T*>(u);
  const T* tp = static_cast<const T*>(table);
  if (vec) gelu_table_kernel<T, E><<<grid, 256, 0, s>>>(up, tp, table_width, vocab, first, tokens, static_cast<T*>(out), rows, W, status);
  else gelu_table_kernel<T, 1><<<grid, 256, 0, s>>>(up, tp, table_width, vocab, first, tokens, static_cast<T*>(out), rows, W, status);
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

extern "C" int b200_poly_norm(const void* z, int64_t row_stride, const float* coef, float eps, void* out, int64_t rows,
                              int32_t width, int32_t dtype, void* stream) {
  using namespace b200;
  if (rows < 0 || width <= 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!z || !coef || !out) return B200_ERR_ARG;
  if (rows > 2147483647) return B200_ERR_TOO_LARGE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = width % E == 0 && row_stride % E == 0 && aligned16(z) && aligned16(out);
  if (dtype == B200_DTYPE_F32) poly_norm<float>(z, row_stride, coef, eps, out, rows, width, vec, s);
  else poly_norm<__nv_bfloat16>(z, row_stride, coef, eps, out, rows, width, vec, s);
  return launch_result();
}

extern "C" int b200_gelu_table(const void* u, const void* table, int64_t table_width, int64_t vocab, int32_t first,
                               const int64_t* tokens, void* out, int64_t rows, int32_t width, int32_t dtype, int32_t* status,
                               void* stream) {
  using namespace b200;
  if (rows < 0 || width <= 0 || first < 0 || first + static_cast<int64_t>(width) > table_width) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!u || !table || !tokens || !out) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) gelu_table<float>(u, table, table_width, vocab, first, tokens, out, rows, width, status, s);
  else gelu_table<__nv_bfloat16>(u, table, table_width, vocab, first, tokens, out, rows, width, status, s);
  return launch_result();
}
