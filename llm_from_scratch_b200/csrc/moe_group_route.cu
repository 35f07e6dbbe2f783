// Expert routing with a choice correction and groups of experts, and the counting sort of the chosen rows by expert:
//
//   s = sigmoid(logits),  c = s + correction,  group score = sum of its two largest c
//   the `top` experts with the largest c inside the `keep` groups with the largest scores
//   weight of a chosen expert = s / (sum of the chosen s + 1e-20)
//
// or, with SOFT, c = logits + correction and the weights are the softmax of c over the chosen experts.
//
// All fp32; equal scores go to the lower index.  A warp per token, the experts of a lane in registers.  Up to kSingle tokens one
// CTA selects and sorts in the same launch; above, a first launch leaves the chosen experts and every CTA's counts, a second
// one places the rows.  Rows of one expert are in no particular order: nothing computed from a row depends on its place.
#include <type_traits>

#include "common.cuh"

namespace b200 {
namespace {

constexpr int kWarps = 8, kSingleWarps = 32, kSingle = 128;
constexpr int kMaxCtas = 128, kMaxExperts = 512, kMaxTop = 32, kMaxGroups = 64;

struct GrArgs {
  const float* logits;       // [T, E]
  const float* correction;   // [E]
  int T, E, K, groups, keep;
  int per_cta;               // tokens per CTA
  int32_t* expert;           // [T, K]
  float* weight;             // [T, K]
  int32_t* offsets;          // [E]
  int32_t* sorted_token;     // [T * K]
  int32_t* slot_to_row;      // [T, K]
  int32_t* counts;           // [CTAs, E]
};

// Writes the token's experts and weights, in order of choice.  EPL: experts per lane, expert e in lane e % 32; `choice`
// [E] and `score` [kMaxGroups] are the warp's.
template <int EPL, bool SOFT>
__device__ __forceinline__ void select_experts(const GrArgs& a, int t, float* choice, float* score) {
  const int lane = threadIdx.x & 31, size = a.E / a.groups;
  float s[EPL], c[EPL];
#pragma unroll
  for (int i = 0; i < EPL; ++i) {
    const int e = lane + 32 * i;
    const float z = e < a.E ? a.logits[static_cast<int64_t>(t) * a.E + e] : 0.f;
    s[i] = SOFT ? z : 1.f / (1.f + expf(-z));
    c[i] = e < a.E ? s[i] + a.correction[e] : -INFINITY;
    if (SOFT) s[i] = c[i];
  }
  if (a.groups > 1) {
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (lane + 32 * i < a.E) choice[lane + 32 * i] = c[i];
    __syncwarp();
    for (int g = lane; g < a.groups; g += 32) {
      float m1 = -INFINITY, m2 = -INFINITY;
      for (int k = 0; k < size; ++k) {
        const float v = choice[g * size + k];
        if (v > m1) {
          m2 = m1;
          m1 = v;
        } else if (v > m2) {
          m2 = v;
        }
      }
      score[g] = size > 1 ? m1 + m2 : m1;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
      const int e = lane + 32 * i;
      if (e >= a.E) continue;
      const int g = e / size;
      const float mine = score[g];
      int better = 0;
      for (int o = 0; o < a.groups; ++o) better += score[o] > mine || (score[o] == mine && o < g);
      if (better >= a.keep) c[i] = -INFINITY;
    }
    __syncwarp();
  }
  unsigned taken = 0;                                  // bit i: this lane's expert i is chosen
  int my_expert = 0;                                   // lane k keeps choice k
  float my_score = 0.f, sum = 0.f, largest = 0.f;      // SOFT: the first choice has the largest score
  for (int k = 0; k < a.K; ++k) {
    float best = -INFINITY;
    int at = kMaxExperts;
#pragma unroll
    for (int i = 0; i < EPL; ++i) {
      const int e = lane + 32 * i;
      if (e < a.E && !(taken >> i & 1) && (at == kMaxExperts || c[i] > best)) {
        best = c[i];
        at = e;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oa = __shfl_xor_sync(0xffffffffu, at, o);
      if (oa != kMaxExperts && (at == kMaxExperts || ob > best || (ob == best && oa < at))) {
        best = ob;
        at = oa;
      }
    }
    float sc = 0.f;
#pragma unroll
    for (int i = 0; i < EPL; ++i)
      if (at == lane + 32 * i) {
        taken |= 1u << i;
        sc = s[i];
      }
    sc = __shfl_sync(0xffffffffu, sc, at & 31);
    if (SOFT) {
      if (k == 0) largest = sc;
      sc = expf(sc - largest);
    }
    if (lane == k) {
      my_expert = at;
      my_score = sc;
    }
    sum += sc;
  }
  if (lane < a.K) {
    a.expert[static_cast<int64_t>(t) * a.K + lane] = my_expert;
    a.weight[static_cast<int64_t>(t) * a.K + lane] = my_score / (SOFT ? sum : sum + 1e-20f);
  }
}

// first output row of every expert into cursor[E] (shared); the caller's totals and the rows of earlier CTAs are in tot / bef
__device__ __forceinline__ void expert_starts(const GrArgs& a, const int32_t* tot, const int32_t* bef, int32_t* cursor, bool write) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int carry = 0;
    for (int e0 = 0; e0 < a.E; e0 += 32) {
      const int e = e0 + lane, v = e < a.E ? tot[e] : 0;
      int x = v;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int y = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x += y;
      }
      if (e < a.E) {
        cursor[e] = carry + x - v + (bef ? bef[e] : 0);
        if (write) a.offsets[e] = carry + x;
      }
      carry += __shfl_sync(0xffffffffu, x, 31);
    }
  }
  __syncthreads();
}

__device__ __forceinline__ void place_rows(const GrArgs& a, int t0, int t1, int32_t* cursor) {
  for (int i = t0 * a.K + threadIdx.x; i < t1 * a.K; i += blockDim.x) {
    const int row = atomicAdd(&cursor[a.expert[i]], 1);
    a.sorted_token[row] = i / a.K;
    a.slot_to_row[i] = row;
  }
}

template <int EPL, bool SINGLE, bool SOFT>
__global__ void __launch_bounds__((SINGLE ? kSingleWarps : kWarps) * 32) group_select_kernel(const GrArgs a) {
  constexpr int W = SINGLE ? kSingleWarps : kWarps;
  extern __shared__ float choices[];                   // [W][E] with groups
  __shared__ float scores[W][kMaxGroups];
  __shared__ int32_t count[EPL * 32], cursor[SINGLE ? EPL * 32 : 1];
  const int warp = threadIdx.x >> 5, t0 = blockIdx.x * a.per_cta, t1 = min(t0 + a.per_cta, a.T);
  for (int e = threadIdx.x; e < EPL * 32; e += blockDim.x) count[e] = 0;
  for (int t = t0 + warp; t < t1; t += W) select_experts<EPL, SOFT>(a, t, choices + warp * a.E, scores[warp]);
  __syncthreads();                                     // the CTA's choices are written, and visible to it
  for (int i = t0 * a.K + threadIdx.x; i < t1 * a.K; i += blockDim.x) atomicAdd(&count[a.expert[i]], 1);
  __syncthreads();
  if constexpr (SINGLE) {
    expert_starts(a, count, nullptr, cursor, true);
    place_rows(a, t0, t1, cursor);
  } else {
    for (int e = threadIdx.x; e < a.E; e += blockDim.x) a.counts[static_cast<int64_t>(blockIdx.x) * a.E + e] = count[e];
  }
}

__global__ void __launch_bounds__(kWarps * 32) group_place_kernel(const GrArgs a) {
  __shared__ int32_t tot[kMaxExperts], bef[kMaxExperts], cursor[kMaxExperts];
  for (int e = threadIdx.x; e < a.E; e += blockDim.x) {
    int sum = 0, before = 0;
    for (unsigned c = 0; c < gridDim.x; ++c) {
      const int v = a.counts[static_cast<int64_t>(c) * a.E + e];
      sum += v;
      if (c < blockIdx.x) before += v;
    }
    tot[e] = sum;
    bef[e] = before;
  }
  __syncthreads();
  expert_starts(a, tot, bef, cursor, blockIdx.x == 0);
  const int t0 = blockIdx.x * a.per_cta;
  place_rows(a, t0, min(t0 + a.per_cta, a.T), cursor);
}

template <int EPL, bool SOFT>
void launch(const GrArgs& a, int ctas, bool single, cudaStream_t s) {
  const size_t per_warp = a.groups > 1 ? a.E * sizeof(float) : 0;
  if (single) {
    group_select_kernel<EPL, true, SOFT><<<1, kSingleWarps * 32, kSingleWarps * per_warp, s>>>(a);
  } else {
    group_select_kernel<EPL, false, SOFT><<<ctas, kWarps * 32, kWarps * per_warp, s>>>(a);
    group_place_kernel<<<ctas, kWarps * 32, 0, s>>>(a);
  }
}

}  // namespace
}  // namespace b200

extern "C" size_t b200_moe_group_route_workspace_bytes(int32_t num_tokens, int32_t num_experts, int32_t top) {
  if (num_tokens <= 0 || num_experts <= 0 || top <= 0) return 0;
  return (static_cast<size_t>(num_tokens) * top + static_cast<size_t>(b200::kMaxCtas) * num_experts) * sizeof(int32_t);
}

namespace b200 {
namespace {
int route(const float* logits, const float* correction, int32_t num_tokens, int32_t num_experts, int32_t top, int32_t groups,
          int32_t keep, bool soft, int32_t* sorted_token, float* weight, int32_t* expert_offsets, int32_t* slot_to_row,
          void* workspace, size_t workspace_bytes, void* stream) {
  if (num_tokens < 0 || num_experts <= 0 || top <= 0 || groups <= 0 || num_experts % groups || keep <= 0 || keep > groups ||
      top > keep * (num_experts / groups))
    return B200_ERR_ARG;
  if (num_experts > kMaxExperts || top > kMaxTop || groups > kMaxGroups) return B200_ERR_UNSUPPORTED;
  if (static_cast<int64_t>(num_tokens) * top > 2147483647LL) return B200_ERR_TOO_LARGE;
  if (num_tokens == 0) return B200_OK;
  if (!logits || !correction || !sorted_token || !weight || !expert_offsets || !slot_to_row) return B200_ERR_ARG;
  if (!workspace || workspace_bytes < b200_moe_group_route_workspace_bytes(num_tokens, num_experts, top))
    return B200_ERR_WORKSPACE;
  GrArgs a{logits, correction, num_tokens, num_experts, top, groups, keep, num_tokens, static_cast<int32_t*>(workspace), weight,
           expert_offsets, sorted_token, slot_to_row, static_cast<int32_t*>(workspace) + static_cast<size_t>(num_tokens) * top};
  int ctas = 1;
  const bool single = num_tokens <= kSingle && num_experts <= 256;      // shared memory: a score row per warp
  if (!single) {
    a.per_cta = (num_tokens + kWarps * kMaxCtas - 1) / (kWarps * kMaxCtas) * kWarps;
    ctas = (num_tokens + a.per_cta - 1) / a.per_cta;
  }
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  auto go = [&](auto epl) {
    if (soft) launch<decltype(epl)::value, true>(a, ctas, single, s);
    else launch<decltype(epl)::value, false>(a, ctas, single, s);
  };
  if (num_experts <= 32) go(std::integral_constant<int, 1>());
  else if (num_experts <= 64) go(std::integral_constant<int, 2>());
  else if (num_experts <= 128) go(std::integral_constant<int, 4>());
  else if (num_experts <= 256) go(std::integral_constant<int, 8>());
  else go(std::integral_constant<int, 16>());
  return launch_result();
}
}  // namespace
}  // namespace b200

extern "C" int b200_moe_group_route(const float* logits, const float* correction, int32_t num_tokens, int32_t num_experts,
                                    int32_t top, int32_t groups, int32_t keep, int32_t* sorted_token, float* weight,
                                    int32_t* expert_offsets, int32_t* slot_to_row, void* workspace, size_t workspace_bytes,
                                    void* stream) {
  return b200::route(logits, correction, num_tokens, num_experts, top, groups, keep, false, sorted_token, weight, expert_offsets,
                     slot_to_row, workspace, workspace_bytes, stream);
}

extern "C" int b200_moe_softmax_route(const float* logits, const float* bias, int32_t num_tokens, int32_t num_experts, int32_t top,
                                      int32_t* sorted_token, float* weight, int32_t* expert_offsets, int32_t* slot_to_row,
                                      void* workspace, size_t workspace_bytes, void* stream) {
  return b200::route(logits, bias, num_tokens, num_experts, top, 1, 1, true, sorted_token, weight, expert_offsets, slot_to_row,
                     workspace, workspace_bytes, stream);
}
