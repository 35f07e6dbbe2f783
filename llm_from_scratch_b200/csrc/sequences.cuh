// Where the tokens, the state slot and the segments of a ragged batch's sequences lie; shared by the kernels that carry
// per-sequence state.  ``Args`` has cu_q / cu_k (or ctx_lens, one token per sequence), slots, num_slots and status.
#pragma once

#include "common.cuh"

namespace b200 {

// The sequence's token range, first position and state slot; false = nothing to do.
struct SeqInfo {
  int64_t tok0;
  int len;
  int64_t pos0;      // position of the first token
  bool fresh;        // it is the first token of the sequence
  int64_t slot;
};
template <typename Args>
__device__ __forceinline__ bool sequence_info(const Args& a, int s, SeqInfo* r) {
  if (a.cu_q != nullptr) {
    r->tok0 = a.cu_q[s];
    r->len = a.cu_q[s + 1] - a.cu_q[s];
    r->pos0 = (a.cu_k[s + 1] - a.cu_k[s]) - r->len;
  } else {
    const int64_t n = a.ctx_lens[s];
    r->tok0 = s;
    r->len = n > 0 ? 1 : 0;
    r->pos0 = n - 1;
  }
  r->fresh = r->pos0 <= 0;
  r->slot = a.slots[s];
  if (r->slot >= a.num_slots) {
    if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
    return false;
  }
  return r->len > 0 && r->slot >= 0;
}

// Segment number -> (sequence, index within it) when every sequence of n is cut into segments of seg_len tokens;
// false: no such segment (index: how many segments behind the last one).  Every thread of the CTA calls it.
__device__ __forceinline__ bool find_segment(const int32_t* cu_q, int n, int seg_len, int number, int* seq, int* index) {
  __shared__ int found[2];
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int left = number, hit_seq = -1, hit_idx = 0;
    for (int base = 0; base < n && hit_seq < 0; base += 32) {
      const int s = base + lane;
      const int t = s < n ? (cu_q[s + 1] - cu_q[s] + seg_len - 1) / seg_len : 0;
      int incl = t;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, incl, o);
        if (lane >= o) incl += y;
      }
      const unsigned hit = __ballot_sync(0xffffffffu, left < incl);
      if (hit) {
        const int src = __ffs(hit) - 1;
        hit_seq = base + src;
        hit_idx = left - __shfl_sync(0xffffffffu, incl - t, src);
      } else {
        left -= __shfl_sync(0xffffffffu, incl, 31);
      }
    }
    if (lane == 0) {
      found[0] = hit_seq;
      found[1] = hit_seq < 0 ? left : hit_idx;
    }
  }
  __syncthreads();
  *seq = found[0];
  *index = found[1];
  return found[0] >= 0;
}

// The tokens of one segment, for kernels that also serve the padding rows behind the last sequence: those form segments of
// their own, in no sequence.
struct Segment {
  int64_t first;     // row of its first token
  int count;
  int index;         // segments of the sequence before it
  int len;           // tokens of the sequence in this step
  int64_t pos0;      // position of the sequence's first token in this step
  int64_t slot;      // of its state, -1: none
};
// The CTA's segment; false: it has none.  ``Args`` as for sequence_info, with n sequences over T rows.  With ctx_lens row i is
// sequence i, one token; else the grid holds T / seg_len + n + 1 CTAs.  Every thread of the CTA calls it.
template <typename Args>
__device__ __forceinline__ bool segment_of(const Args& a, int seg_len, Segment* r) {
  if (a.cu_q == nullptr) {
    r->first = blockIdx.x;
    r->count = r->len = 1;
    r->index = 0;
    r->pos0 = a.ctx_lens ? max(a.ctx_lens[blockIdx.x] - 1, static_cast<int64_t>(0)) : 0;
    r->slot = a.ctx_lens && a.slots && a.ctx_lens[blockIdx.x] > 0 ? a.slots[blockIdx.x] : -1;
  } else {
    int seq;
    if (find_segment(a.cu_q, a.n, seg_len, blockIdx.x, &seq, &r->index)) {
      const int q0 = a.cu_q[seq];
      r->len = a.cu_q[seq + 1] - q0;
      r->first = q0 + static_cast<int64_t>(r->index) * seg_len;
      r->count = min(seg_len, r->len - r->index * seg_len);
      r->pos0 = (a.cu_k[seq + 1] - a.cu_k[seq]) - r->len;
      r->slot = a.slots ? a.slots[seq] : -1;
    } else {
      r->first = a.cu_q[a.n] + static_cast<int64_t>(r->index) * seg_len;
      if (r->first >= a.T) return false;
      r->count = static_cast<int>(a.T - r->first < seg_len ? a.T - r->first : seg_len);
      r->len = r->count;
      r->index = 0;
      r->pos0 = 0;
      r->slot = -1;
    }
  }
  if (r->slot >= a.num_slots) {
    if (threadIdx.x == 0) report(a.status, B200_ERR_BOUNDS);
    r->slot = -1;
  }
  return true;
}

// Number of the first segment of sequence seq.  Threads of warp 0 call it.
__device__ __forceinline__ int first_segment(const int32_t* cu_q, int seg_len, int seq) {
  int sum = 0;
  for (int s = threadIdx.x & 31; s < seq; s += 32) sum += (cu_q[s + 1] - cu_q[s] + seg_len - 1) / seg_len;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  return sum;
}

// ---- packed fp32 pairs ----
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// ---- scalar functions of gates (one exponential, one approximate reciprocal of 1 ulp) ----
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// sigmoid(z) and sigmoid(-z) from one exponential of -|z|, so that the small one keeps its relative accuracy
__device__ __forceinline__ void sigmoids(float z, float* s, float* s_neg) {
  const float t = expf(-fabsf(z)), big = rcp_approx(1.f + t), small = t * big;
  *s = z >= 0.f ? big : small;
  *s_neg = z >= 0.f ? small : big;
}
__device__ __forceinline__ float sigmoid_f(float x) {
  float s, n;
  sigmoids(x, &s, &n);
  return s;
}
__device__ __forceinline__ float silu_f(float x) { return x * sigmoid_f(x); }
// for values that are rounded to T next: in bf16 on the approximate exponential (relative error below 2^-20)
template <typename T>
__device__ __forceinline__ float sigmoid_for(float x) {
  return sizeof(T) == 2 ? rcp_approx(1.f + fast_exp2(-1.4426950408889634f * x)) : sigmoid_f(x);
}
template <typename T>
__device__ __forceinline__ float silu_for(float x) { return x * sigmoid_for<T>(x); }

}  // namespace b200
