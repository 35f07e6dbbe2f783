// Gated residual of a decoder whose sublayers run side by side on one input: every sublayer's result passes an element-wise
// gate on its way into the fp32 residual, and the step that combines a token's experts is part of the same launch:
//
//   x <- x + y1 sigmoid(g1) + y2 sigmoid(g2),   h = x in the activation dtype
//   y2[t] = sum_k weight[t, k] rows[slot[t, k]]    when the second sublayer is a mixture of experts
//
// Sums, gates and weights are fp32.
#include "sequences.cuh"

namespace b200 {
namespace {

struct GrArgs {
  float* x;                  // [T, d]
  const void* y1;            // [T, d]
  const void* g1;            // [T, d], row stride g_stride
  const void* y2;            // [T, d], or expert rows [T * top_k, d]; null: one sublayer
  const void* g2;
  int64_t g_stride;
  const float* weight;       // [T, top_k]
  const int32_t* slot;       // [T, top_k]
  int top_k;                 // 0: y2 holds one row per token
  void* h;                   // [T, d]
  int64_t T;
  int d;
  int32_t* status;
};

template <typename T, int E>
struct Vals {
  float v[E];
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (E > 1) {
      union {
        uint4 u;
        T e[16 / sizeof(T)];
      } k;
      k.u = *reinterpret_cast<const uint4*>(p);
#pragma unroll
      for (int i = 0; i < E; ++i) v[i] = to_float<T>(k.e[i]);
    } else {
      v[0] = to_float<T>(p[0]);
    }
  }
};

// E elements (16 bytes) per access, or one
template <typename T, int E>
__global__ void __launch_bounds__(256) gated_residual_kernel(const GrArgs a) {
  const int64_t units = a.d / E, total = a.T * units;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<int64_t>(gridDim.x) * blockDim.x) {
    const int64_t t = i / units;
    const int c = static_cast<int>(i - t * units) * E;
    float* xp = a.x + t * a.d + c;
    float x[E];
    if constexpr (E >= 4) {
#pragma unroll
      for (int e = 0; e < E; e += 4) {
        const float4 v = *reinterpret_cast<const float4*>(xp + e);
        x[e] = v.x, x[e + 1] = v.y, x[e + 2] = v.z, x[e + 3] = v.w;
      }
    } else {
      x[0] = xp[0];
    }
    Vals<T, E> y, g;
    y.load(static_cast<const T*>(a.y1) + t * a.d + c);
    g.load(static_cast<const T*>(a.g1) + t * a.g_stride + c);
    if (a.y2 != nullptr) {
      Vals<T, E> y2, g2;
      g2.load(static_cast<const T*>(a.g2) + t * a.g_stride + c);
      if (a.top_k == 0) {
        y2.load(static_cast<const T*>(a.y2) + t * a.d + c);
      } else {
#pragma unroll
        for (int e = 0; e < E; ++e) y2.v[e] = 0.f;
        for (int k = 0; k < a.top_k; ++k) {
          const int row = a.slot[t * a.top_k + k];
          const float w = a.weight[t * a.top_k + k];
          if (row < 0 || row >= a.T * a.top_k) {
            report(a.status, B200_ERR_BOUNDS);
            continue;
          }
          Vals<T, E> r;
          r.load(static_cast<const T*>(a.y2) + static_cast<int64_t>(row) * a.d + c);
#pragma unroll
          for (int e = 0; e < E; ++e) y2.v[e] += w * r.v[e];
        }
      }
#pragma unroll
      for (int e = 0; e < E; ++e) x[e] += y2.v[e] * sigmoid_f(g2.v[e]);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) x[e] += y.v[e] * sigmoid_f(g.v[e]);
    T* hp = static_cast<T*>(a.h) + t * a.d + c;
    if constexpr (E >= 4) {
      union {
        uint4 u;
        T e[16 / sizeof(T)];
      } o;
#pragma unroll
      for (int e = 0; e < E; ++e) o.e[e] = from_float<T>(x[e]);
#pragma unroll
      for (int e = 0; e < E; e += 4) *reinterpret_cast<float4*>(xp + e) = make_float4(x[e], x[e + 1], x[e + 2], x[e + 3]);
      *reinterpret_cast<uint4*>(hp) = o.u;
    } else {
      xp[0] = x[0];
      hp[0] = from_float<T>(x[0]);
    }
  }
}

template <typename T>
void launch(const GrArgs& a, bool vec, cudaStream_t s) {
  constexpr int E = 16 / sizeof(T);
  const int64_t blocks = (a.T * (a.d / (vec ? E : 1)) + 255) / 256;
  const unsigned grid = static_cast<unsigned>(blocks < 148 * 64 ? blocks : 148 * 64);
  if (vec) gated_residual_kernel<T, E><<<grid, 256, 0, s>>>(a);
  else gated_residual_kernel<T, 1><<<grid, 256, 0, s>>>(a);
}

}  // namespace
}  // namespace b200

extern "C" int b200_gated_residual(float* x, const void* y1, const void* gate1, const void* y2, const void* gate2,
                                   int64_t gate_stride, const float* row_weight, const int32_t* slot_to_row, int32_t top_k,
                                   void* h, int64_t rows, int32_t d, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (rows < 0 || d <= 0 || top_k < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!x || !y1 || !gate1 || !h || (y2 && !gate2) || (top_k > 0 && (!y2 || !row_weight || !slot_to_row))) return B200_ERR_ARG;
  GrArgs a{x, y1, gate1, y2, gate2, gate_stride, row_weight, slot_to_row, top_k, h, rows, d, status};
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = d % E == 0 && gate_stride % E == 0 && aligned16(x) && aligned16(y1) && aligned16(gate1) && aligned16(h) &&
                   (!y2 || (aligned16(y2) && aligned16(gate2)));
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B200_DTYPE_F32) launch<float>(a, vec, s);
  else launch<__nv_bfloat16>(a, vec, s);
  return launch_result();
}
