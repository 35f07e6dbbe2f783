// Rows of a latent key/value cache without a rotary part: the norm of the down-projection with its scatter into the
// paged pool, and the gather of whole contexts back out of the pool for the prefill expansion.
#include "sequences.cuh"

namespace b200 {
namespace {

constexpr int kWarps = 8;

struct LnArgs {
  const void* in;            // [T, r] (token stride free)
  int64_t stride;
  const float* w;            // [r]
  float eps;
  void* out;                 // [T, r]
  void* cache;               // [slots, r] or null
  const int64_t* slots;
  int64_t num_slots, T;
  int r;
  int32_t* status;
};

// a warp per row; E elements per 16-byte access, or one
template <typename T, int E>
__global__ void __launch_bounds__(kWarps * 32) latent_norm_kernel(const LnArgs a) {
  const int lane = threadIdx.x & 31;
  const int64_t t = static_cast<int64_t>(blockIdx.x) * kWarps + (threadIdx.x >> 5);
  if (t >= a.T) return;
  const T* src = static_cast<const T*>(a.in) + t * a.stride;
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  float ss = 0.f;
  for (int c = lane * E; c < a.r; c += 32 * E) {
    if constexpr (E > 1) {
      Pack p;
      p.u = *reinterpret_cast<const uint4*>(src + c);
#pragma unroll
      for (int i = 0; i < E; ++i) ss += to_float<T>(p.e[i]) * to_float<T>(p.e[i]);
    } else {
      ss += to_float<T>(src[c]) * to_float<T>(src[c]);
    }
  }
  const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(a.r) + a.eps);
  int64_t slot = a.cache ? a.slots[t] : -1;
  if (slot >= a.num_slots) {
    if (lane == 0) report(a.status, B200_ERR_BOUNDS);
    slot = -1;
  }
  T* out = static_cast<T*>(a.out) + t * a.r;
  T* pool = slot >= 0 ? static_cast<T*>(a.cache) + slot * a.r : nullptr;
  for (int c = lane * E; c < a.r; c += 32 * E) {
    if constexpr (E > 1) {
      Pack p, o;
      p.u = *reinterpret_cast<const uint4*>(src + c);
#pragma unroll
      for (int i = 0; i < E; ++i) o.e[i] = from_float<T>(to_float<T>(p.e[i]) * inv * a.w[c + i]);
      *reinterpret_cast<uint4*>(out + c) = o.u;
      if (pool) *reinterpret_cast<uint4*>(pool + c) = o.u;
    } else {
      const T o = from_float<T>(to_float<T>(src[c]) * inv * a.w[c]);
      out[c] = o;
      if (pool) pool[c] = o;
    }
  }
}

struct GaArgs {
  const void* cache;         // [num_blocks, bs, W]
  const int32_t* bt;
  int64_t bt_stride;
  int bs;
  int64_t num_blocks;
  const int32_t* cu_k;       // [n + 1]
  void* out;                 // [rows, W]
  int64_t rows;
  int W;                     // row width in units
  int32_t* status;
};

// rows of sequence blockIdx.y, a warp per row; U is the copy unit
template <typename U>
__global__ void __launch_bounds__(kWarps * 32) gather_rows_kernel(const GaArgs a) {
  const int s = blockIdx.y, lane = threadIdx.x & 31;
  const int k0 = a.cu_k[s], len = a.cu_k[s + 1] - k0;
  const int64_t base = k0 - a.cu_k[0];
  for (int j = blockIdx.x * kWarps + (threadIdx.x >> 5); j < len; j += gridDim.x * kWarps) {
    const int blk = j / a.bs;
    int64_t id = -1;
    if (blk < a.bt_stride) id = a.bt[s * a.bt_stride + blk];
    if (id < 0 || id >= a.num_blocks || base + j >= a.rows) {
      if (lane == 0) report(a.status, B200_ERR_BOUNDS);
      continue;
    }
    const U* src = static_cast<const U*>(a.cache) + (id * a.bs + j % a.bs) * a.W;
    U* dst = static_cast<U*>(a.out) + (base + j) * a.W;
    for (int c = lane; c < a.W; c += 32) dst[c] = src[c];
  }
}

// out = o * sigmoid(g), element by element; o contiguous [T, W], g [T, W] with a row stride; a CTA per row
template <typename T, int E>
__global__ void __launch_bounds__(256) sigmoid_gate_kernel(T* o, const T* g, int64_t g_stride, int W) {
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  o += static_cast<int64_t>(blockIdx.x) * W;
  g += blockIdx.x * g_stride;
  for (int c = threadIdx.x * E; c < W; c += blockDim.x * E) {
    if constexpr (E > 1) {
      Pack a, b;
      a.u = *reinterpret_cast<const uint4*>(o + c);
      b.u = *reinterpret_cast<const uint4*>(g + c);
#pragma unroll
      for (int k = 0; k < E; ++k) a.e[k] = from_float<T>(to_float<T>(a.e[k]) * sigmoid_for<T>(to_float<T>(b.e[k])));
      *reinterpret_cast<uint4*>(o + c) = a.u;
    } else {
      o[c] = from_float<T>(to_float<T>(o[c]) * sigmoid_for<T>(to_float<T>(g[c])));
    }
  }
}

}  // namespace
}  // namespace b200

extern "C" int b200_latent_norm_store(const void* rows_in, int64_t in_stride, const float* norm_w, float eps, void* rows_out,
                                      void* cache, const int64_t* slot_mapping, int64_t num_slots, int64_t num_tokens,
                                      int32_t rank, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_tokens < 0 || rank <= 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_tokens == 0) return B200_OK;
  if (!rows_in || !norm_w || !rows_out || (cache && !slot_mapping)) return B200_ERR_ARG;
  if (num_tokens > 2147483647LL * kWarps) return B200_ERR_TOO_LARGE;
  LnArgs a{rows_in, in_stride, norm_w, eps, rows_out, cache, slot_mapping, num_slots, num_tokens, rank, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const unsigned grid = static_cast<unsigned>((num_tokens + kWarps - 1) / kWarps);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = rank % E == 0 && in_stride % E == 0 && aligned16(rows_in) && aligned16(rows_out) && (!cache || aligned16(cache));
  if (dtype == B200_DTYPE_F32) {
    if (vec) latent_norm_kernel<float, 4><<<grid, kWarps * 32, 0, s>>>(a);
    else latent_norm_kernel<float, 1><<<grid, kWarps * 32, 0, s>>>(a);
  } else {
    if (vec) latent_norm_kernel<__nv_bfloat16, 8><<<grid, kWarps * 32, 0, s>>>(a);
    else latent_norm_kernel<__nv_bfloat16, 1><<<grid, kWarps * 32, 0, s>>>(a);
  }
  return launch_result();
}

extern "C" int b200_gather_rows(const void* cache, int32_t block_size, int64_t num_blocks, int64_t row_bytes,
                                const int32_t* block_tables, int64_t bt_stride, const int32_t* cu_seqlens_k,
                                int32_t num_seqs, int32_t max_seqlen_k, void* out, int64_t out_rows, int32_t* status,
                                void* stream) {
  using namespace b200;
  if (block_size <= 0 || num_blocks <= 0 || row_bytes <= 0 || bt_stride <= 0 || num_seqs < 0 || max_seqlen_k < 0)
    return B200_ERR_ARG;
  if (num_seqs == 0 || max_seqlen_k == 0) return B200_OK;
  if (!cache || !block_tables || !cu_seqlens_k || !out) return B200_ERR_ARG;
  if (num_seqs > 65535 || row_bytes % 2) return B200_ERR_UNSUPPORTED;
  GaArgs a{cache, block_tables, bt_stride, block_size, num_blocks, cu_seqlens_k, out, out_rows, 0, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid((max_seqlen_k + 4 * kWarps - 1) / (4 * kWarps), num_seqs);
  if (row_bytes % 16 == 0 && aligned16(cache) && aligned16(out)) {
    a.W = static_cast<int>(row_bytes / 16);
    gather_rows_kernel<uint4><<<grid, kWarps * 32, 0, s>>>(a);
  } else {
    a.W = static_cast<int>(row_bytes / 2);
    gather_rows_kernel<uint16_t><<<grid, kWarps * 32, 0, s>>>(a);
  }
  return launch_result();
}

extern "C" int b200_sigmoid_gate(void* o, const void* gate, int64_t gate_stride, int64_t rows, int32_t width, int32_t dtype,
                                 void* stream) {
  using namespace b200;
  if (rows < 0 || width <= 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!o || !gate) return B200_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = width % E == 0 && gate_stride % E == 0 && aligned16(o) && aligned16(gate);
  if (rows > 2147483647) return B200_ERR_TOO_LARGE;
  const int units = (width + (vec ? E : 1) - 1) / (vec ? E : 1), threads = units >= 256 ? 256 : (units + 31) / 32 * 32;
  const unsigned grid = static_cast<unsigned>(rows);
  if (dtype == B200_DTYPE_F32) {
    auto* p = static_cast<float*>(o);
    auto* g = static_cast<const float*>(gate);
    if (vec) sigmoid_gate_kernel<float, 4><<<grid, threads, 0, s>>>(p, g, gate_stride, width);
    else sigmoid_gate_kernel<float, 1><<<grid, threads, 0, s>>>(p, g, gate_stride, width);
  } else {
    auto* p = static_cast<__nv_bfloat16*>(o);
    auto* g = static_cast<const __nv_bfloat16*>(gate);
    if (vec) sigmoid_gate_kernel<__nv_bfloat16, 8><<<grid, threads, 0, s>>>(p, g, gate_stride, width);
    else sigmoid_gate_kernel<__nv_bfloat16, 1><<<grid, threads, 0, s>>>(p, g, gate_stride, width);
  }
  return launch_result();
}
