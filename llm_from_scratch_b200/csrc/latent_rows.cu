// Rows of a latent key/value cache: the norm of the down-projection (with the rotation of a rotary part behind it, and the
// norm of a query latent beside it) with its scatter into the paged pool, the rotation of the queries' rotary channels, and
// the gather of contexts, or of the ends of contexts, back out of the pool for the prefill expansion.
#include "rotary.cuh"
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

struct LpArgs {
  const void* q_in;          // [T, rq] query latents (row stride free) or null
  int64_t q_stride;
  const float* wq;           // [rq]
  int rq;
  void* q_out;               // [T, rq]
  const void* kv_in;         // [T, r + dr]
  int64_t kv_stride;
  const float* wkv;          // [r]
  int r, dr;
  float eps;
  const double* freq;        // [half]
  int half;                  // rotated pairs, the first of the rotary part
  float magnitude;           // of cos and sin
  const int64_t* positions;  // [T]
  void* kv_out;              // [T, r + dr]
  void* cache;               // [slots, r + dr] or null
  const int64_t* slots;
  int64_t num_slots, T;
  int32_t* status;
};

// dst (and dst2, if given) = src / rms(src) * w over n elements, by a warp; E elements per access.  Rows of up to kKeep
// accesses per lane stay in registers between the two passes.
constexpr int kKeep = 4;
template <typename T, int E>
__device__ __forceinline__ void warp_norm(const T* src, const float* w, int n, float eps, T* dst, T* dst2) {
  const int lane = threadIdx.x & 31;
  union Pack {
    uint4 u;
    T e[16 / sizeof(T)];
  };
  auto load = [&](int c) {
    Pack p;
    if constexpr (E > 1) p.u = *reinterpret_cast<const uint4*>(src + c);
    else p.e[0] = src[c];
    return p;
  };
  Pack keep[kKeep];
  float ss = 0.f;
  auto add = [&](const Pack& p) {
#pragma unroll
    for (int i = 0; i < E; ++i) ss += to_float<T>(p.e[i]) * to_float<T>(p.e[i]);
  };
#pragma unroll
  for (int k = 0; k < kKeep; ++k)
    if ((k * 32 + lane) * E < n) keep[k] = load((k * 32 + lane) * E);
#pragma unroll
  for (int k = 0; k < kKeep; ++k)
    if ((k * 32 + lane) * E < n) add(keep[k]);
  for (int c = (kKeep * 32 + lane) * E; c < n; c += 32 * E) add(load(c));
  const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(n) + eps);
  auto put = [&](int c, Pack p) {
    if constexpr (E > 1) {
#pragma unroll
      for (int i = 0; i < E; i += 4) {
        const float4 wv = *reinterpret_cast<const float4*>(w + c + i);
        p.e[i] = from_float<T>(to_float<T>(p.e[i]) * inv * wv.x);
        p.e[i + 1] = from_float<T>(to_float<T>(p.e[i + 1]) * inv * wv.y);
        p.e[i + 2] = from_float<T>(to_float<T>(p.e[i + 2]) * inv * wv.z);
        p.e[i + 3] = from_float<T>(to_float<T>(p.e[i + 3]) * inv * wv.w);
      }
      *reinterpret_cast<uint4*>(dst + c) = p.u;
      if (dst2) *reinterpret_cast<uint4*>(dst2 + c) = p.u;
    } else {
      p.e[0] = from_float<T>(to_float<T>(p.e[0]) * inv * w[c]);
      dst[c] = p.e[0];
      if (dst2) dst2[c] = p.e[0];
    }
  };
#pragma unroll
  for (int k = 0; k < kKeep; ++k)
    if ((k * 32 + lane) * E < n) put((k * 32 + lane) * E, keep[k]);
  for (int c = (kKeep * 32 + lane) * E; c < n; c += 32 * E) put(c, load(c));
}

// blockIdx.y 0: latent rows; 1: query latents.  A warp per row; EQ / EK elements per access
template <typename T, int EQ, int EK>
__global__ void __launch_bounds__(kWarps * 32) latent_prologue_kernel(const LpArgs a) {
  const int lane = threadIdx.x & 31;
  const int64_t t = static_cast<int64_t>(blockIdx.x) * kWarps + (threadIdx.x >> 5);
  if (t >= a.T) return;
  if (blockIdx.y == 1) {
    warp_norm<T, EQ>(static_cast<const T*>(a.q_in) + t * a.q_stride, a.wq, a.rq, a.eps, static_cast<T*>(a.q_out) + t * a.rq,
                     nullptr);
    return;
  }
  const int W = a.r + a.dr;
  int64_t slot = a.cache ? a.slots[t] : -1;
  if (slot >= a.num_slots) {
    if (lane == 0) report(a.status, B200_ERR_BOUNDS);
    slot = -1;
  }
  const T* src = static_cast<const T*>(a.kv_in) + t * a.kv_stride;
  T* out = static_cast<T*>(a.kv_out) + t * W;
  T* pool = slot >= 0 ? static_cast<T*>(a.cache) + slot * W : nullptr;
  const int64_t pos = a.positions[t];
  for (int i = lane; 2 * i < a.dr; i += 32) {
    const int c = a.r + 2 * i;
    const bool pair = 2 * i + 1 < a.dr;
    float u = to_float<T>(src[c]), v = pair ? to_float<T>(src[c + 1]) : 0.f;
    if (i < a.half) {
      const float2 cs = rotary_angle(pos, a.freq[i]);
      const float co = cs.x * a.magnitude, si = cs.y * a.magnitude, nu = u * co - v * si;
      v = v * co + u * si;
      u = nu;
    }
    out[c] = from_float<T>(u);
    if (pair) out[c + 1] = from_float<T>(v);
    if (pool) {
      pool[c] = from_float<T>(u);
      if (pair) pool[c + 1] = from_float<T>(v);
    }
  }
  warp_norm<T, EK>(src, a.wkv, a.r, a.eps, out, pool);
}

struct RtArgs {
  void* q;                   // [T, H, D], in place
  int64_t T;
  int H, D, dr;              // the last dr channels of a head are its rotary part
  const double* freq;
  int half;
  float magnitude;
  const int64_t* positions;
  void* tail;                // [tail_rows, H, dr] or null: a copy of the rotated parts of the first rows
  int64_t tail_rows;
  int per_cta;               // tokens
};

// per_cta tokens per CTA; V consecutive channels (whole pairs, 16 bytes) per thread and trip, or one pair
template <typename T, int V>
__global__ void __launch_bounds__(256) rotate_heads_kernel(const RtArgs a) {
  extern __shared__ float2 cs[];     // [per_cta][half]
  const int64_t t0 = static_cast<int64_t>(blockIdx.x) * a.per_cta;
  const int nt = static_cast<int>(a.T - t0 < a.per_cta ? a.T - t0 : a.per_cta);
  for (int i = threadIdx.x; i < nt * a.half; i += blockDim.x) {
    const int t = i / a.half, j = i - t * a.half;
    const float2 r = rotary_angle(a.positions[t0 + t], a.freq[j]);
    cs[i] = make_float2(r.x * a.magnitude, r.y * a.magnitude);
  }
  __syncthreads();
  constexpr int W = V > 2 ? V : 2;
  const int units = (a.dr + W - 1) / W, per = a.H * units;
  for (int i = threadIdx.x; i < nt * per; i += blockDim.x) {
    const int t = i / per, k = i - t * per, h = k / units, c = (k - h * units) * W;
    const int64_t tok = t0 + t;
    T* p = static_cast<T*>(a.q) + (tok * a.H + h) * a.D + (a.D - a.dr) + c;
    T* tail = tok < a.tail_rows ? static_cast<T*>(a.tail) + (tok * a.H + h) * a.dr + c : nullptr;
    float x[W];
    union {
      uint4 u;
      T e[16 / sizeof(T)];
    } pack;
    const bool pair = c + 1 < a.dr;
    if constexpr (V > 2) {
      pack.u = *reinterpret_cast<const uint4*>(p);
#pragma unroll
      for (int e = 0; e < W; ++e) x[e] = to_float<T>(pack.e[e]);
    } else {
      x[0] = to_float<T>(p[0]);
      x[1] = pair ? to_float<T>(p[1]) : 0.f;
    }
#pragma unroll
    for (int e = 0; e < W; e += 2) {
      const int j = (c + e) >> 1;
      if (j < a.half) {
        const float2 r = cs[t * a.half + j];
        const float u = x[e], v = x[e + 1];
        x[e] = u * r.x - v * r.y;
        x[e + 1] = v * r.x + u * r.y;
      }
    }
    if constexpr (V > 2) {
#pragma unroll
      for (int e = 0; e < W; ++e) pack.e[e] = from_float<T>(x[e]);
      *reinterpret_cast<uint4*>(p) = pack.u;
      if (tail) *reinterpret_cast<uint4*>(tail) = pack.u;
    } else {
      p[0] = from_float<T>(x[0]);
      if (pair) p[1] = from_float<T>(x[1]);
      if (tail) {
        tail[0] = from_float<T>(x[0]);
        if (pair) tail[1] = from_float<T>(x[1]);
      }
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
  const int32_t* cu_full;    // [n + 1] or null: whole contexts, of which cu_k counts the last rows
  void* out;                 // [rows, W]
  int64_t rows;
  int W;                     // row width in units
  int n;                     // sequences
  int32_t* status;
};

// rows of sequence blockIdx.y, a warp per row; U is the copy unit.  blockIdx.y == n: zeros behind the last row
template <typename U>
__global__ void __launch_bounds__(kWarps * 32) gather_rows_kernel(const GaArgs a) {
  const int s = blockIdx.y, lane = threadIdx.x & 31;
  if (s == a.n) {
    for (int64_t j = a.cu_k[s] - a.cu_k[0] + blockIdx.x * kWarps + (threadIdx.x >> 5); j < a.rows; j += gridDim.x * kWarps)
      for (int c = lane; c < a.W; c += 32) static_cast<U*>(a.out)[j * a.W + c] = U{};
    return;
  }
  const int k0 = a.cu_k[s], len = a.cu_k[s + 1] - k0;
  const int64_t base = k0 - a.cu_k[0];
  const int skip = a.cu_full ? max(a.cu_full[s + 1] - a.cu_full[s] - len, 0) : 0;
  for (int j = blockIdx.x * kWarps + (threadIdx.x >> 5); j < len; j += gridDim.x * kWarps) {
    const int pos = skip + j, blk = pos / a.bs;
    int64_t id = -1;
    if (blk < a.bt_stride) id = a.bt[s * a.bt_stride + blk];
    if (id < 0 || id >= a.num_blocks || base + j >= a.rows) {
      if (lane == 0) report(a.status, B200_ERR_BOUNDS);
      continue;
    }
    const U* src = static_cast<const U*>(a.cache) + (id * a.bs + pos % a.bs) * a.W;
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
  return b200_gather_last_rows(cache, block_size, num_blocks, row_bytes, block_tables, bt_stride, cu_seqlens_k, nullptr,
                               num_seqs, max_seqlen_k, out, out_rows, status, stream);
}

extern "C" int b200_gather_last_rows(const void* cache, int32_t block_size, int64_t num_blocks, int64_t row_bytes,
                                     const int32_t* block_tables, int64_t bt_stride, const int32_t* cu_seqlens_k,
                                     const int32_t* cu_seqlens_full, int32_t num_seqs, int32_t max_seqlen_k, void* out,
                                     int64_t out_rows, int32_t* status, void* stream) {
  using namespace b200;
  if (block_size <= 0 || num_blocks <= 0 || row_bytes <= 0 || bt_stride <= 0 || num_seqs < 0 || max_seqlen_k < 0)
    return B200_ERR_ARG;
  if (num_seqs == 0 || max_seqlen_k == 0) return B200_OK;
  if (!cache || !block_tables || !cu_seqlens_k || !out) return B200_ERR_ARG;
  if (num_seqs >= 65535 || row_bytes % 2) return B200_ERR_UNSUPPORTED;
  GaArgs a{cache, block_tables, bt_stride, block_size, num_blocks, cu_seqlens_k, cu_seqlens_full, out, out_rows, 0, num_seqs, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid((max_seqlen_k + 4 * kWarps - 1) / (4 * kWarps), num_seqs + 1);
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

extern "C" int b200_latent_prologue(const void* q_in, int64_t q_stride, const float* q_norm_w, int32_t q_rank, void* q_out,
                                    const void* kv_in, int64_t kv_stride, const float* kv_norm_w, int32_t kv_rank,
                                    int32_t rope_dim, float eps, const double* freq, int32_t rot_dims, float magnitude,
                                    const int64_t* positions, void* kv_out, void* cache, const int64_t* slot_mapping,
                                    int64_t num_slots, int64_t num_tokens, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (num_tokens < 0 || kv_rank <= 0 || rope_dim < 0 || rot_dims < 0 || rot_dims % 2 || rot_dims > rope_dim || (q_in && q_rank <= 0))
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_tokens == 0) return B200_OK;
  if (!kv_in || !kv_norm_w || !kv_out || !positions || (rot_dims > 0 && !freq) || (q_in && (!q_norm_w || !q_out)) ||
      (cache && !slot_mapping))
    return B200_ERR_ARG;
  if (num_tokens > 2147483647LL * kWarps) return B200_ERR_TOO_LARGE;
  LpArgs a{q_in, q_stride, q_norm_w, q_rank, q_out, kv_in, kv_stride, kv_norm_w, kv_rank, rope_dim, eps, freq, rot_dims / 2,
           magnitude, positions, kv_out, cache, slot_mapping, num_slots, num_tokens, status};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>((num_tokens + kWarps - 1) / kWarps), q_in ? 2 : 1);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vq = !q_in || (q_rank % E == 0 && q_stride % E == 0 && aligned16(q_in) && aligned16(q_out) && aligned16(q_norm_w));
  const bool vk = kv_rank % E == 0 && (kv_rank + rope_dim) % E == 0 && kv_stride % E == 0 && aligned16(kv_in) && aligned16(kv_out) &&
                  aligned16(kv_norm_w) && (!cache || aligned16(cache));
  if (dtype == B200_DTYPE_F32) {
    if (vq && vk) latent_prologue_kernel<float, 4, 4><<<grid, kWarps * 32, 0, s>>>(a);
    else latent_prologue_kernel<float, 1, 1><<<grid, kWarps * 32, 0, s>>>(a);
  } else {
    if (vq && vk) latent_prologue_kernel<__nv_bfloat16, 8, 8><<<grid, kWarps * 32, 0, s>>>(a);
    else latent_prologue_kernel<__nv_bfloat16, 1, 1><<<grid, kWarps * 32, 0, s>>>(a);
  }
  return launch_result();
}

extern "C" int b200_rotate_heads(void* q, int64_t num_tokens, int32_t num_heads, int32_t head_dim, int32_t rope_dim,
                                 const double* freq, int32_t rot_dims, float magnitude, const int64_t* positions, void* tail,
                                 int64_t tail_rows, int32_t dtype, void* stream) {
  using namespace b200;
  if (num_tokens < 0 || num_heads <= 0 || rope_dim < 0 || rope_dim > head_dim || rot_dims < 0 || rot_dims % 2 ||
      rot_dims > rope_dim || tail_rows < 0 || tail_rows > num_tokens)
    return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (num_tokens == 0 || rope_dim == 0) return B200_OK;
  if (!q || !positions || (rot_dims > 0 && !freq) || (tail_rows > 0 && !tail)) return B200_ERR_ARG;
  if (rot_dims > 2048 || num_tokens > 2147483647LL) return B200_ERR_UNSUPPORTED;
  RtArgs a{q, num_tokens, num_heads, head_dim, rope_dim, freq, rot_dims / 2, magnitude, positions, tail, tail_rows, 1};
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  // a few tokens per CTA share its threads for their angles; small steps spread over the SMs instead
  a.per_cta = num_tokens >= 4096 ? 4 : num_tokens >= 512 ? 2 : 1;
  const unsigned grid = static_cast<unsigned>((num_tokens + a.per_cta - 1) / a.per_cta);
  const size_t smem = sizeof(float2) * a.per_cta * (rot_dims / 2);
  const int E = dtype == B200_DTYPE_F32 ? 4 : 8;
  const bool vec = head_dim % E == 0 && rope_dim % E == 0 && aligned16(q) && (!tail || aligned16(tail));
  if (dtype == B200_DTYPE_F32) {
    if (vec) rotate_heads_kernel<float, 4><<<grid, 256, smem, s>>>(a);
    else rotate_heads_kernel<float, 2><<<grid, 256, smem, s>>>(a);
  } else {
    if (vec) rotate_heads_kernel<__nv_bfloat16, 8><<<grid, 256, smem, s>>>(a);
    else rotate_heads_kernel<__nv_bfloat16, 2><<<grid, 256, smem, s>>>(a);
  }
  return launch_result();
}
