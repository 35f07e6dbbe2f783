// fp32 residual of a decoder that norms what a sublayer gives, with one number per norm, and mixes neighbouring tokens on the way
// into the next mixer.  One launch per boundary between sublayers:
//
//   x' = x + gain y / sqrt(mean(y^2) + eps)        y: the sublayer's result, or the weighted sum of a token's expert rows
//   x' = scale embed[token]                        (the first boundary)
//   h  = x' + (before - x') shift                  before: the previous token's x' (its sequence's state slot when that token came
//                                                  in an earlier step, zeros ahead of the first token)
//   h  = final_gain x' / sqrt(mean(x'^2) + eps)    or
//   h  = x', rounded to the activation dtype
//
// x' goes to a buffer of its own: with a shift a CTA also needs the row before its first one, and works it out once more from x
// and y, which the row's own CTA must not have overwritten.  A CTA owns up to R rows of one sequence.  The CTA that reads a
// sequence's state is the one that moves it on: it works out the sequence's last row, if that is not its own.
#include <initializer_list>

#include "sequences.cuh"

namespace b200 {
namespace {

struct ShArgs {
  const float* x;            // [T, d], unused with embed
  float* x_out;              // [T, d] or null
  const int64_t* tokens;     // [T] with embed
  const void* embed;         // [vocab, d] or null
  int64_t vocab;
  float scale;               // of the embedding row
  const void* y;             // [T, d], or expert rows [T * top, d]
  const float* weight;       // [T, top]
  const int32_t* row_of;     // [T, top]
  int top;                   // 0: y holds one row per token
  float gain;
  const float* shift;        // [d] or null
  float* state;              // [slots, d]
  const int64_t* slots;      // [n]
  int64_t num_slots;
  const int32_t* cu_q;       // [n + 1], or null: row i is sequence i
  const int32_t* cu_k;
  const int64_t* ctx_lens;
  int n;
  int norm;                  // h is the final norm
  float final_gain, eps;
  void* h;                   // [T, d]
  int64_t T;
  int d;
  int32_t* status;
};

// V channels in fp32
template <typename T, int V>
__device__ __forceinline__ void load_row(const T* p, float (&v)[V]) {
  if constexpr (V * sizeof(T) % 16 == 0) {
    union {
      uint4 u;
      T e[16 / sizeof(T)];
    } k;
#pragma unroll
    for (int i = 0; i < V; i += 16 / sizeof(T)) {
      k.u = *reinterpret_cast<const uint4*>(p + i);
#pragma unroll
      for (int j = 0; j < static_cast<int>(16 / sizeof(T)); ++j) v[i + j] = to_float<T>(k.e[j]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_float<T>(p[i]);
  }
}
template <typename T, int V>
__device__ __forceinline__ void store_row(T* p, const float (&v)[V]) {
  if constexpr (V * sizeof(T) % 16 == 0) {
    union {
      uint4 u;
      T e[16 / sizeof(T)];
    } k;
#pragma unroll
    for (int i = 0; i < V; i += 16 / sizeof(T)) {
#pragma unroll
      for (int j = 0; j < static_cast<int>(16 / sizeof(T)); ++j) k.e[j] = from_float<T>(v[i + j]);
      *reinterpret_cast<uint4*>(p + i) = k.u;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = from_float<T>(v[i]);
  }
}

// y of channels c .. c + V - 1 of a row
template <typename T, int V>
__device__ __forceinline__ void load_y(const ShArgs& a, int64_t row, int c, float (&y)[V]) {
  if (a.top == 0) {
    load_row<T, V>(static_cast<const T*>(a.y) + row * a.d + c, y);
    return;
  }
#pragma unroll
  for (int i = 0; i < V; ++i) y[i] = 0.f;
#pragma unroll 4
  for (int k = 0; k < a.top; ++k) {
    const int from = a.row_of[row * a.top + k];
    const float w = a.weight[row * a.top + k];
    if (from < 0 || from >= a.T * a.top) {
      report(a.status, B200_ERR_BOUNDS);
      continue;
    }
    float r[V];
    load_row<T, V>(static_cast<const T*>(a.y) + static_cast<int64_t>(from) * a.d + c, r);
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] += w * r[i];
  }
}

// x of channels c .. before y joins
template <typename T, int V>
__device__ __forceinline__ void load_x(const ShArgs& a, int64_t row, int c, float (&x)[V]) {
  if (a.embed == nullptr) {
    load_row<float, V>(a.x + row * a.d + c, x);
    return;
  }
  int64_t tok = a.tokens[row];
  if (tok < 0 || tok >= a.vocab) {
    if (c == 0) report(a.status, B200_ERR_BOUNDS);
    tok = 0;
  }
  load_row<T, V>(static_cast<const T*>(a.embed) + tok * a.d + c, x);
#pragma unroll
  for (int i = 0; i < V; ++i) x[i] *= a.scale;
}

// Sums over the CTA of N values per thread; scratch [N][32].
template <int N>
__device__ __forceinline__ void cta_sums(float (&v)[N], float (*scratch)[32]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
  for (int j = 0; j < N; ++j) v[j] = warp_sum(v[j]);
  if (lane == 0) {
#pragma unroll
    for (int j = 0; j < N; ++j) scratch[j][warp] = v[j];
  }
  __syncthreads();
#pragma unroll
  for (int j = 0; j < N; ++j) v[j] = warp_sum(lane < nw ? scratch[j][lane] : 0.f);
}

// The rows of a CTA: own ones first .. first + count - 1, and at most one more row that is worked out and not written: the row
// before them, or the sequence's last one for its state.
struct Work {
  Segment g;
  int64_t extra;             // row or -1
  bool halo;                 // extra is the row before
  bool from_state, save;
};
template <bool SHIFT>
__device__ __forceinline__ bool work_of(const ShArgs& a, int rows, Work* w) {
  w->extra = -1;
  w->halo = w->from_state = w->save = false;
  if constexpr (SHIFT) {
    if (!segment_of(a, rows, &w->g)) return false;
    const Segment& g = w->g;
    if (g.index > 0) {
      w->halo = true;
      w->extra = g.first - 1;
    } else {
      w->save = g.slot >= 0;
      w->from_state = w->save && g.pos0 > 0;
      if (w->save && g.len > g.count) w->extra = g.first + g.len - 1;
    }
  } else {
    w->g.first = static_cast<int64_t>(blockIdx.x) * rows;
    w->g.count = static_cast<int>(a.T - w->g.first < rows ? a.T - w->g.first : rows);
    w->g.slot = -1;
  }
  return true;
}

// V channels per thread, all of a row in one pass
template <typename T, int V, int R, bool SHIFT>
__global__ void __launch_bounds__(R > 1 ? 512 : 1024) shift_residual_kernel(const ShArgs a) {
  constexpr int N = SHIFT ? R + 1 : R;                 // row R: the extra one
  __shared__ float scratch[2][N][32];
  Work w;
  if (!work_of<SHIFT>(a, R, &w)) return;
  const int c = threadIdx.x * V;
  const bool in = c < a.d;
  float x[N][V], y[N][V], ss[N];
  auto row = [&](int j) -> int64_t { return j < R ? (j < w.g.count ? w.g.first + j : -1) : w.extra; };
#pragma unroll
  for (int j = 0; j < N; ++j) {
    ss[j] = 0.f;
#pragma unroll
    for (int i = 0; i < V; ++i) x[j][i] = y[j][i] = 0.f;
    if (!in || row(j) < 0) continue;
    load_x<T, V>(a, row(j), c, x[j]);
    if (a.y != nullptr) load_y<T, V>(a, row(j), c, y[j]);
  }
  float carried[V], mix[V];
  if constexpr (SHIFT) {
#pragma unroll
    for (int i = 0; i < V; ++i) carried[i] = mix[i] = 0.f;
    if (in) {
      load_row<float, V>(a.shift + c, mix);
      if (w.from_state) load_row<float, V>(a.state + w.g.slot * a.d + c, carried);
    }
  }
  if (a.y != nullptr) {
#pragma unroll
    for (int j = 0; j < N; ++j)
#pragma unroll
      for (int i = 0; i < V; ++i) ss[j] += y[j][i] * y[j][i];
    cta_sums<N>(ss, scratch[0]);
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const float f = a.gain * rsqrtf(ss[j] / static_cast<float>(a.d) + a.eps);
#pragma unroll
      for (int i = 0; i < V; ++i) x[j][i] += f * y[j][i];
    }
  }
  if (a.x_out != nullptr && in) {
#pragma unroll
    for (int j = 0; j < R; ++j)
      if (j < w.g.count) store_row<float, V>(a.x_out + row(j) * a.d + c, x[j]);
  }
  T* h = static_cast<T*>(a.h) + c;
  if constexpr (SHIFT) {
    if (!in) return;
    if (w.halo) {
#pragma unroll
      for (int i = 0; i < V; ++i) carried[i] = x[R][i];
    }
#pragma unroll
    for (int j = 0; j < R; ++j) {
      if (j >= w.g.count) break;
      float o[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        o[i] = x[j][i] + (carried[i] - x[j][i]) * mix[i];
        carried[i] = x[j][i];
      }
      store_row<T, V>(h + row(j) * a.d, o);
    }
    if (w.save) {
      if (w.extra >= 0) {
#pragma unroll
        for (int i = 0; i < V; ++i) carried[i] = x[R][i];
      }
      store_row<float, V>(a.state + w.g.slot * a.d + c, carried);
    }
  } else {
    if (a.norm) {
#pragma unroll
      for (int j = 0; j < N; ++j) {
        ss[j] = 0.f;
#pragma unroll
        for (int i = 0; i < V; ++i) ss[j] += x[j][i] * x[j][i];
      }
      cta_sums<N>(ss, scratch[1]);
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const float f = a.final_gain * rsqrtf(ss[j] / static_cast<float>(a.d) + a.eps);
#pragma unroll
        for (int i = 0; i < V; ++i) x[j][i] *= f;
      }
    }
    if (!in) return;
#pragma unroll
    for (int j = 0; j < R; ++j)
      if (j < w.g.count) store_row<T, V>(h + row(j) * a.d, x[j]);
  }
}

// any width, a row per CTA
template <typename T, bool SHIFT>
__global__ void __launch_bounds__(256) shift_residual_any_kernel(const ShArgs a) {
  __shared__ float scratch[2][2][32];
  Work w;
  if (!work_of<SHIFT>(a, 1, &w)) return;
  const int64_t row = w.g.first;
  float ss[2] = {0.f, 0.f};
  if (a.y != nullptr) {
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
      float y[1];
      load_y<T, 1>(a, row, c, y);
      ss[0] += y[0] * y[0];
      if (w.extra >= 0) {
        load_y<T, 1>(a, w.extra, c, y);
        ss[1] += y[0] * y[0];
      }
    }
    cta_sums<2>(ss, scratch[0]);
  }
  const float f0 = a.gain * rsqrtf(ss[0] / static_cast<float>(a.d) + a.eps);
  const float f1 = a.gain * rsqrtf(ss[1] / static_cast<float>(a.d) + a.eps);
  auto value = [&](int64_t r, int c, float f) -> float {
    float x[1], y[1] = {0.f};
    load_x<T, 1>(a, r, c, x);
    if (a.y != nullptr) load_y<T, 1>(a, r, c, y);
    return x[0] + f * y[0];
  };
  T* h = static_cast<T*>(a.h) + row * a.d;
  float sq[2] = {0.f, 0.f};
  for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
    const float x = value(row, c, f0);
    if (a.x_out != nullptr) a.x_out[row * a.d + c] = x;
    if constexpr (SHIFT) {
      const float extra = w.extra >= 0 ? value(w.extra, c, f1) : 0.f;
      const float before = w.halo ? extra : w.from_state ? a.state[w.g.slot * a.d + c] : 0.f;
      h[c] = from_float<T>(x + (before - x) * a.shift[c]);
      if (w.save) a.state[w.g.slot * a.d + c] = w.extra >= 0 ? extra : x;
    } else {
      sq[0] += x * x;
      if (!a.norm) h[c] = from_float<T>(x);
    }
  }
  if constexpr (!SHIFT) {
    if (!a.norm) return;
    cta_sums<2>(sq, scratch[1]);
    const float f = a.final_gain * rsqrtf(sq[0] / static_cast<float>(a.d) + a.eps);
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) h[c] = from_float<T>(value(row, c, f0) * f);
  }
}

constexpr int kRows = 4;             // rows per CTA of prompts
constexpr int64_t kManyRows = 2048;  // below, a CTA per row fills the GPU better

template <typename T, bool SHIFT>
void launch(const ShArgs& a, bool vec, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const int threads = (a.d / V + 31) / 32 * 32;
  const bool one_each = SHIFT && a.cu_q == nullptr;
  auto grid = [&](int rows) {
    if (one_each) return static_cast<unsigned>(a.T);
    if (SHIFT) return static_cast<unsigned>(a.T / rows + a.n + 1);
    return static_cast<unsigned>((a.T + rows - 1) / rows);
  };
  if (!vec || threads > 1024) shift_residual_any_kernel<T, SHIFT><<<grid(1), 256, 0, s>>>(a);
  else if (a.T >= kManyRows && threads <= 512 && !one_each) shift_residual_kernel<T, V, kRows, SHIFT><<<grid(kRows), threads, 0, s>>>(a);
  else shift_residual_kernel<T, V, 1, SHIFT><<<grid(1), threads, 0, s>>>(a);
}

}  // namespace
}  // namespace b200

extern "C" int b200_shift_residual(const float* x, float* x_out, const int64_t* tokens, const void* embed, int64_t vocab,
                                   float embed_scale, const void* y, const float* row_weight, const int32_t* slot_to_row,
                                   int32_t top, float gain, const float* shift, float* state, int64_t num_slots,
                                   const int64_t* state_slots, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                   const int64_t* context_lens, int32_t num_seqs, int32_t final_norm, float final_gain, float eps,
                                   void* h, int64_t rows, int32_t d, int32_t dtype, int32_t* status, void* stream) {
  using namespace b200;
  if (rows < 0 || d <= 0 || top < 0 || num_slots < 0 || num_seqs < 0) return B200_ERR_ARG;
  if (dtype != B200_DTYPE_F32 && dtype != B200_DTYPE_BF16) return B200_ERR_UNSUPPORTED;
  if (rows == 0) return B200_OK;
  if (!h || (embed ? !tokens : !x) || (top > 0 && (!y || !row_weight || !slot_to_row))) return B200_ERR_ARG;
  if (shift) {
    if (!state || !state_slots || final_norm || x == x_out) return B200_ERR_ARG;
    if (cu_seqlens_q ? !cu_seqlens_k : !context_lens) return B200_ERR_ARG;
    if (!cu_seqlens_q && num_seqs != rows) return B200_ERR_ARG;
  }
  if (rows > 2147483647 - num_seqs) return B200_ERR_TOO_LARGE;
  ShArgs a{x, x_out, tokens, embed, vocab, embed_scale, y, row_weight, slot_to_row, top, gain, shift, state, state_slots,
           num_slots, cu_seqlens_q, cu_seqlens_k, context_lens, num_seqs, final_norm, final_gain, eps, h, rows, d, status};
  const int V = dtype == B200_DTYPE_F32 ? 4 : 8;
  bool vec = d % V == 0;
  for (const void* p : {static_cast<const void*>(x), static_cast<const void*>(x_out), embed, y, static_cast<const void*>(shift),
                        static_cast<const void*>(state), static_cast<const void*>(h)})
    vec = vec && aligned16(p);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto t) {
    using T = decltype(t);
    if (shift) launch<T, true>(a, vec, s);
    else launch<T, false>(a, vec, s);
  };
  if (dtype == B200_DTYPE_F32) go(float());
  else go(__nv_bfloat16());
  return launch_result();
}
