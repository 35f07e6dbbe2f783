// Pieces shared by the gated delta rule's kernels: arguments and the scalar gates of a (token, head).
#pragma once

#include "sequences.cuh"

namespace b200 {

struct DeltaArgs {
  // q, k [T, G, dk], v [T, H, dv] behind convolution and silu (token stride act_stride), or, where the step kernel does
  // the convolution itself, the raw projections (act_stride = proj_stride)
  const void* q;
  const void* k;
  const void* v;
  int64_t act_stride;
  const void* b;             // [T, H] write strength before the sigmoid
  const void* a;             // [T, H] decay input
  const void* gate;          // [T, H, dv] output gate before silu
  int64_t proj_stride;       // of b, a, gate
  const float* dt_bias;      // [H]
  const float* a_log;        // [H]
  const float* norm_w;       // [dv]
  float eps;
  float* state;              // [slots, H, dk, dv]
  const int64_t* slots;      // [n], < 0: skip the sequence
  int64_t num_slots;
  const int32_t* cu_q;       // [n + 1], or null: one token per sequence
  const int32_t* cu_k;       // [n + 1] with cu_q
  const int64_t* ctx_lens;   // [n] without cu_q
  void* out;                 // [T, H, dv]
  int n, H, G, dk, dv;
  // convolution of the step kernel: weights [taps, conv_width], ring [slots, taps, conv_width]; column of q / k / v
  const float* conv_w;
  float* conv_ring;
  int taps, conv_width, col_q, col_k, col_v;
  int32_t* status;
};

// write strength beta = sigmoid(b) and ln g = -exp(a_log) softplus(a + dt_bias)
__device__ __forceinline__ float log_decay(float z, float a_log) {
  const float sp = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
  return -expf(a_log) * sp;
}

// prompts and portions on tensor cores (delta_chunk.cu): bf16, dk and dv multiples of 16 up to 128
bool delta_chunk_shape(int dk, int dv);
size_t delta_chunk_workspace(int num_seqs, int64_t total_tokens, int H);
int delta_chunk_launch(const DeltaArgs& a, int64_t total_tokens, void* workspace, cudaStream_t s);

}  // namespace b200
