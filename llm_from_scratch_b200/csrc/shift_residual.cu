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
// and y, which the row's own CTA must not have overwritten.  A CTA walks up to `rows` rows of one sequence in order, the next
// row's loads in flight while it reduces and writes the current one; the row before stays in registers.  The CTA that reads a
// sequence's state is the one that moves it on: it also works out the sequence's last row, if that is not its own.
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
  int rows;                  // rows per CTA, at most kMaxRows
};

constexpr int kMaxRows = 8;

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

// Sum over the CTA; scratch is of this use alone until the next barrier but one.
__device__ __forceinline__ float cta_sum(float v, float* scratch) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  v = warp_sum(v);
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? scratch[lane] : 0.f);
}

// The rows of a CTA: own ones first .. first + count - 1, and at most one more row that is worked out and not written: the row
// before them (halo), or the sequence's last one for its state (tail).
struct Work {
  Segment g;
  bool halo, tail, from_state, save;
  // rows in the order of the walk
  __device__ __forceinline__ int steps() const { return g.count + halo + tail; }
  __device__ __forceinline__ int64_t row(int i) const {
    return tail && i == g.count ? g.first + g.len - 1 : g.first + i - halo;
  }
  __device__ __forceinline__ bool own(int i) const { return i >= halo && i < g.count + halo; }
};
template <bool SHIFT>
__device__ __forceinline__ bool work_of(const ShArgs& a, int rows, Work* w) {
  w->halo = w->tail = w->from_state = w->save = false;
  if constexpr (SHIFT) {
    if (!segment_of(a, rows, &w->g)) return false;
    const Segment& g = w->g;
    w->halo = g.index > 0;
    w->save = g.index == 0 && g.slot >= 0;
    w->from_state = w->save && g.pos0 > 0;
    w->tail = w->save && g.len > g.count;
  } else {
    w->g.first = static_cast<int64_t>(blockIdx.x) * rows;
    w->g.count = static_cast<int>(a.T - w->g.first < rows ? a.T - w->g.first : rows);
  }
  return true;
}

// What is loaded of a row ahead of its turn: x, and y as it lies in memory (TOP > 0: one piece per expert).
template <typename T, int V, int TOP>
struct Ahead {
  float x[V];
  uint4 y[TOP > 0 ? TOP : 1];
};

// V channels per thread (16 bytes of T), a row in one pass.  TOP: 0: y holds one row per token, else at most TOP expert rows
template <typename T, int TOP, bool SHIFT>
__global__ void __launch_bounds__(1024) shift_residual_kernel(const ShArgs a) {
  constexpr int V = 16 / sizeof(T);
  __shared__ float scratch[2][32], scratch_norm[2][32];
  __shared__ int s_from[(kMaxRows + 1) * (TOP > 0 ? TOP : 1)];
  __shared__ float s_weight[(kMaxRows + 1) * (TOP > 0 ? TOP : 1)];
  Work w;
  if (!work_of<SHIFT>(a, a.rows, &w)) return;
  const int c = threadIdx.x * V, steps = w.steps();
  const bool in = c < a.d;
  if constexpr (TOP > 0) {
    for (int i = threadIdx.x; i < steps * TOP; i += blockDim.x) {
      const int k = i % TOP;
      int from = -1;
      float weight = 0.f;
      if (k < a.top) {
        const int64_t at = w.row(i / TOP) * a.top + k;
        from = a.row_of[at];
        weight = a.weight[at];
        if (from < 0 || from >= a.T * a.top) {
          report(a.status, B200_ERR_BOUNDS);
          from = -1;
        }
      }
      s_from[i] = from;
      s_weight[i] = weight;
    }
    __syncthreads();
  }
  auto fetch = [&](int i, Ahead<T, V, TOP>& r) {
    if (!in) return;
    const int64_t row = w.row(i);
    load_x<T, V>(a, row, c, r.x);
    if constexpr (TOP > 0) {
#pragma unroll
      for (int k = 0; k < TOP; ++k) {
        const int from = s_from[i * TOP + k];
        r.y[k] = from < 0 ? make_uint4(0, 0, 0, 0)
                          : *reinterpret_cast<const uint4*>(static_cast<const T*>(a.y) + static_cast<int64_t>(from) * a.d + c);
      }
    } else if (a.y != nullptr) {
      r.y[0] = *reinterpret_cast<const uint4*>(static_cast<const T*>(a.y) + row * a.d + c);
    }
  };
  auto unpack = [&](uint4 u, float (&v)[V]) {
    union {
      uint4 u;
      T e[V];
    } k;
    k.u = u;
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_float<T>(k.e[i]);
  };
  float before[V];
  if constexpr (SHIFT) {
#pragma unroll
    for (int i = 0; i < V; ++i) before[i] = 0.f;
    if (in && w.from_state) load_row<float, V>(a.state + w.g.slot * a.d + c, before);
  }
  Ahead<T, V, TOP> next;
#pragma unroll
  for (int i = 0; i < V; ++i) next.x[i] = 0.f;
#pragma unroll
  for (int k = 0; k < (TOP > 0 ? TOP : 1); ++k) next.y[k] = make_uint4(0, 0, 0, 0);
  fetch(0, next);
  for (int i = 0; i < steps; ++i) {
    float x[V], y[V];
    if constexpr (TOP > 0) {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
#pragma unroll
      for (int k = 0; k < TOP; ++k) {
        float r[V];
        unpack(next.y[k], r);
        const float f = s_weight[i * TOP + k];
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(f, r[e], y[e]);
      }
    } else {
      unpack(next.y[0], y);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = next.x[e];
    if (i + 1 < steps) fetch(i + 1, next);
    if (a.y != nullptr) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) ss += y[e] * y[e];
      const float f = a.gain * rsqrtf(cta_sum(ss, scratch[i & 1]) / static_cast<float>(a.d) + a.eps);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] += f * y[e];
    }
    const int64_t row = w.row(i);
    T* h = static_cast<T*>(a.h) + row * a.d + c;
    const bool own = w.own(i);
    if (own && in && a.x_out != nullptr) store_row<float, V>(a.x_out + row * a.d + c, x);
    if constexpr (SHIFT) {
      if (own && in) {
        float mix[V];
        load_row<float, V>(a.shift + c, mix);
#pragma unroll
        for (int e = 0; e < V; ++e) mix[e] = x[e] + (before[e] - x[e]) * mix[e];
        store_row<T, V>(h, mix);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) before[e] = x[e];
    } else {
      if (a.norm) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) ss += x[e] * x[e];
        const float f = a.final_gain * rsqrtf(cta_sum(ss, scratch_norm[i & 1]) / static_cast<float>(a.d) + a.eps);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] *= f;
      }
      if (in) store_row<T, V>(h, x);
    }
  }
  if constexpr (SHIFT) {
    if (w.save && in) store_row<float, V>(a.state + w.g.slot * a.d + c, before);      // the last row of the walk is the sequence's
  }
}

// any width, a row per CTA
template <typename T, bool SHIFT>
__global__ void __launch_bounds__(256) shift_residual_any_kernel(const ShArgs a) {
  __shared__ float scratch[3][32];
  Work w;
  if (!work_of<SHIFT>(a, 1, &w)) return;
  const int64_t row = w.g.first, extra = w.halo ? row - 1 : w.tail ? row + w.g.len - 1 : -1;
  float s0 = 0.f, s1 = 0.f;
  if (a.y != nullptr) {
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
      float y[1];
      load_y<T, 1>(a, row, c, y);
      s0 += y[0] * y[0];
      if (extra >= 0) {
        load_y<T, 1>(a, extra, c, y);
        s1 += y[0] * y[0];
      }
    }
    s0 = cta_sum(s0, scratch[0]);
    s1 = cta_sum(s1, scratch[1]);
  }
  const float f0 = a.gain * rsqrtf(s0 / static_cast<float>(a.d) + a.eps);
  const float f1 = a.gain * rsqrtf(s1 / static_cast<float>(a.d) + a.eps);
  auto value = [&](int64_t r, int c, float f) -> float {
    float x[1], y[1] = {0.f};
    load_x<T, 1>(a, r, c, x);
    if (a.y != nullptr) load_y<T, 1>(a, r, c, y);
    return x[0] + f * y[0];
  };
  T* h = static_cast<T*>(a.h) + row * a.d;
  float sq = 0.f;
  for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
    const float x = value(row, c, f0);
    sq += x * x;
    if constexpr (SHIFT) {
      const float other = extra >= 0 ? value(extra, c, f1) : 0.f;
      const float before = w.halo ? other : w.from_state ? a.state[w.g.slot * a.d + c] : 0.f;
      h[c] = from_float<T>(x + (before - x) * a.shift[c]);
      if (w.save) a.state[w.g.slot * a.d + c] = w.tail ? other : x;
      if (a.x_out != nullptr) a.x_out[row * a.d + c] = x;
    } else if (!a.norm) {
      h[c] = from_float<T>(x);
      if (a.x_out != nullptr) a.x_out[row * a.d + c] = x;
    }
  }
  if constexpr (!SHIFT) {
    if (!a.norm) return;
    const float f = a.final_gain * rsqrtf(cta_sum(sq, scratch[2]) / static_cast<float>(a.d) + a.eps);
    for (int c = threadIdx.x; c < a.d; c += blockDim.x) {
      const float x = value(row, c, f0);
      if (a.x_out != nullptr) a.x_out[row * a.d + c] = x;
      h[c] = from_float<T>(x * f);
    }
  }
}

template <typename T, bool SHIFT>
void launch(ShArgs a, bool vec, cudaStream_t s) {
  constexpr int V = 16 / sizeof(T);
  const int threads = (a.d / V + 31) / 32 * 32;
  const bool one_each = SHIFT && a.cu_q == nullptr;
  // long walks save rows that are worked out twice and keep loads in flight; short ones fill the GPU with few rows
  a.rows = one_each ? 1 : a.T >= 148 * 16 ? kMaxRows : a.T >= 148 * 4 ? 2 : 1;
  const bool any = !vec || threads > 1024 || a.top > 8;
  if (any) a.rows = 1;
  const unsigned grid = static_cast<unsigned>(one_each ? a.T : SHIFT ? a.T / a.rows + a.n + 1 : (a.T + a.rows - 1) / a.rows);
  if (any) shift_residual_any_kernel<T, SHIFT><<<grid, 256, 0, s>>>(a);
  else if (a.top == 0) shift_residual_kernel<T, 0, SHIFT><<<grid, threads, 0, s>>>(a);
  else if (a.top <= 2) shift_residual_kernel<T, 2, SHIFT><<<grid, threads, 0, s>>>(a);
  else if (a.top <= 4) shift_residual_kernel<T, 4, SHIFT><<<grid, threads, 0, s>>>(a);
  else shift_residual_kernel<T, 8, SHIFT><<<grid, threads, 0, s>>>(a);
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
           num_slots, cu_seqlens_q, cu_seqlens_k, context_lens, num_seqs, final_norm, final_gain, eps, h, rows, d, status, 1};
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
