// fp32 residual of a decoder, one launch per boundary between sublayers or layers:
//
//   x <- x + y / sqrt(mean(y^2) + eps) * w        y: the sublayer's result, activation dtype (optional)
//   x <- x + scale embed[token]                   (optional; or x starts as that)
//   h  = x, rounded to the activation dtype       what the next sublayer reads, or with a norm
//   h  = x / sqrt(mean(x^2) + eps) * norm_w       mean over the row, or over each of `groups` equal parts of it
//
// One CTA per token row; the row stays in registers, and its loads precede the first reduction.  Weights are read where they
// are used: every CTA of an SM reads the same ones, and without them two CTAs of the widest rows fit an SM.
#include "common.cuh"

namespace b200 {
namespace {

struct ResArgs {
  float* x;                  // [T, d]
  const int64_t* tokens;     // [T] with embed, else null
  const void* embed;         // [vocab, d] or null
  int64_t vocab;
  float scale;               // of the embedding row
  int start;                 // x is not read: it begins as zero
  const void* y;             // [T, d] or null
  const float* w;            // [d]
  const float* final_w;      // [d] or null
  int groups;                // parts of the final norm, a divisor of d
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

constexpr int kMaxParts = 64;      // groups of the final norm in the register kernel
enum Parts { kWhole, kWarps, kAny };

// N groups of four channels per thread, d a multiple of four.  PARTS: the final norm is one part, or a.groups parts of which
// each is whole warps wide (a multiple of 128 channels: one barrier) or any multiple of four channels wide
template <typename T, int N, Parts PARTS>
__global__ void __launch_bounds__(1024, N == 1 ? 2 : 1) residual_norm_kernel(const ResArgs a) {
  __shared__ float scratch[2][32];
  __shared__ float part[PARTS == kAny ? 1024 * N : 32 * N], part_inv[PARTS == kAny ? kMaxParts : 1];
  const int d = a.d, step = blockDim.x * 4, first = threadIdx.x * 4;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * d;
  T* hr = static_cast<T*>(a.h) + row * d;
  float4 x[N], y[N];
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const T* er = a.embed ? static_cast<const T*>(a.embed) + embed_row(a, row) * d : nullptr;
  const T* yr = static_cast<const T*>(a.y) + row * d;
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = first + i * step;
    const bool in = c < d;
    x[i] = in && !a.start ? *reinterpret_cast<const float4*>(xr + c) : zero;
    y[i] = in && a.y ? load4<T>(yr + c) : zero;
  }
  if (a.embed != nullptr) {
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + i * step;
      const float4 e = c < d ? load4<T>(er + c) : zero;
      x[i].x += a.scale * e.x;
      x[i].y += a.scale * e.y;
      x[i].z += a.scale * e.z;
      x[i].w += a.scale * e.w;
    }
  }
  if (a.y != nullptr) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) ss += sumsq(y[i]);
    const float inv = rsqrtf(cta_sum(ss, scratch[0]) / static_cast<float>(d) + a.eps);
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + i * step;
      const float4 w = c < d ? *reinterpret_cast<const float4*>(a.w + c) : zero;
      x[i].x += y[i].x * inv * w.x;
      x[i].y += y[i].y * inv * w.y;
      x[i].z += y[i].z * inv * w.z;
      x[i].w += y[i].w * inv * w.w;
    }
  }
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const int c = first + i * step;
    if (c < d) *reinterpret_cast<float4*>(xr + c) = x[i];
  }
  if (a.final_w != nullptr) {
    float inv[N];
    if constexpr (PARTS == kWarps) {
      const int width = d / a.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const float ss = warp_sum(sumsq(x[i]));
        if (lane == 0) part[i * nw + warp] = ss;              // of channels (i * nw + warp) * 128 ...
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int per = width >> 7, first_warp = (i * nw + warp) / per * per;
        float ss = 0.f;
        for (int k = lane; k < per; k += 32) ss += first_warp + k < N * nw ? part[first_warp + k] : 0.f;
        inv[i] = rsqrtf(warp_sum(ss) / static_cast<float>(width) + a.eps);
      }
    } else if constexpr (PARTS == kAny) {
      const int width = d / a.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        const int c = first + i * step;
        if (c < d) part[c >> 2] = sumsq(x[i]);
      }
      __syncthreads();
      for (int g = warp; g < a.groups; g += blockDim.x >> 5) {
        float ss = 0.f;
        for (int k = lane; k < width >> 2; k += 32) ss += part[g * (width >> 2) + k];
        ss = warp_sum(ss);
        if (lane == 0) part_inv[g] = rsqrtf(ss / static_cast<float>(width) + a.eps);
      }
      __syncthreads();
#pragma unroll
      for (int i = 0; i < N; ++i) inv[i] = part_inv[min((first + i * step) / width, a.groups - 1)];
    } else {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < N; ++i) ss += sumsq(x[i]);
      inv[0] = rsqrtf(cta_sum(ss, scratch[1]) / static_cast<float>(d) + a.eps);
#pragma unroll
      for (int i = 1; i < N; ++i) inv[i] = inv[0];
    }
#pragma unroll
    for (int i = 0; i < N; ++i) {
      const int c = first + i * step;
      const float4 w = c < d ? *reinterpret_cast<const float4*>(a.final_w + c) : zero;
      x[i] = make_float4(x[i].x * inv[i] * w.x, x[i].y * inv[i] * w.y, x[i].z * inv[i] * w.z, x[i].w * inv[i] * w.w);
    }
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
  __shared__ float scratch[32];
  const int d = a.d;
  const int64_t row = blockIdx.x;
  float* xr = a.x + row * d;
  T* hr = static_cast<T*>(a.h) + row * d;
  const T* er = a.embed ? static_cast<const T*>(a.embed) + embed_row(a, row) * d : nullptr;
  const T* yr = a.y ? static_cast<const T*>(a.y) + row * d : nullptr;
  float inv = 0.f;
  if (yr != nullptr) {
    float ss = 0.f;
    for (int c = threadIdx.x; c < d; c += blockDim.x) ss += to_float<T>(yr[c]) * to_float<T>(yr[c]);
    inv = rsqrtf(cta_sum(ss, scratch) / static_cast<float>(d) + a.eps);
  }
  for (int c = threadIdx.x; c < d; c += blockDim.x) {
    float x = a.start ? 0.f : xr[c];
    if (er != nullptr) x += a.scale * to_float<T>(er[c]);
    if (yr != nullptr) x += to_float<T>(yr[c]) * inv * a.w[c];
    xr[c] = x;
    if (a.final_w == nullptr) hr[c] = from_float<T>(x);
  }
  if (a.final_w == nullptr) return;
  __syncthreads();
  const int width = d / a.groups, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int g = warp; g < a.groups; g += blockDim.x >> 5) {     // a warp per part
    float ss = 0.f;
    for (int c = g * width + lane; c < (g + 1) * width; c += 32) ss += xr[c] * xr[c];
    const float r = rsqrtf(warp_sum(ss) / static_cast<float>(width) + a.eps);
    for (int c = g * width + lane; c < (g + 1) * width; c += 32) hr[c] = from_float<T>(xr[c] * r * a.final_w[c]);
  }
}

template <typename T, Parts PARTS>
void launch_vec(const ResArgs& a, unsigned grid, cudaStream_t s) {
  const int groups = a.d / 4;
  if (groups <= 1024) residual_norm_kernel<T, 1, PARTS><<<grid, (groups + 31) / 32 * 32, 0, s>>>(a);
  else residual_norm_kernel<T, 2, PARTS><<<grid, (groups + 63) / 64 * 32, 0, s>>>(a);
}

template <typename T>
void launch(const ResArgs& a, int64_t rows, bool vec, cudaStream_t s) {
  const unsigned grid = static_cast<unsigned>(rows);
  const bool grouped = a.final_w && a.groups > 1;
  if (!vec || a.d / 4 > 2048 || (grouped && (a.d / a.groups % 4 != 0 || a.groups > kMaxParts)))
    residual_norm_any_kernel<T><<<grid, 256, 0, s>>>(a);
  else if (!grouped) launch_vec<T, kWhole>(a, grid, s);
  else if (a.d / a.groups % 128 == 0) launch_vec<T, kWarps>(a, grid, s);
  else launch_vec<T, kAny>(a, grid, s);
}

int residual_norm(const ResArgs& a, int64_t rows, int32_t dtype, void* stream) {
  if (rows < 0 || a.d <= 0 || a.groups <= 0 || a.d % a.groups) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!a.x || !a.h || (a.embed && !a.tokens) || (a.y && !a.w) || (a.start && !a.embed)) return B200_ERR_ARG;
  if (rows > 2147483647) return B200_ERR_TOO_LARGE;
  const bool vec = a.d % 4 == 0 && aligned16(a.x) && aligned16(a.h) && (!a.embed || aligned16(a.embed)) &&
                   (!a.y || (aligned16(a.y) && aligned16(a.w))) && (!a.final_w || aligned16(a.final_w));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) launch<float>(a, rows, vec, s);
  else launch<__nv_bfloat16>(a, rows, vec, s);
  return launch_result();
}

}  // namespace
}  // namespace b200

extern "C" int b200_residual_norm(float* x, const int64_t* tokens, const void* embed, int64_t vocab, const void* y,
                                  const float* norm_w, const float* final_w, float eps, void* h, int64_t rows, int32_t d,
                                  int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (rows > 0 && !embed && !y) return B200_ERR_ARG;
  return residual_norm({x, tokens, embed, vocab, 1.f, embed != nullptr, embed ? nullptr : y, norm_w, final_w, 1, eps, h, d, status},
                       rows, dtype, stream);
}

extern "C" int b200_residual_group_norm(float* x, const void* y, const float* y_norm_w, const int64_t* tokens, const void* embed,
                                        int64_t vocab, float embed_scale, int32_t start, const float* norm_w, int32_t groups,
                                        float eps, void* h, int64_t rows, int32_t d, int32_t dtype, int32_t* status,
                                        void* stream) {
  using namespace b200;
  return residual_norm({x, tokens, embed, vocab, embed_scale, start != 0, y, y_norm_w, norm_w, groups, eps, h, d, status}, rows,
                       dtype, stream);
}
