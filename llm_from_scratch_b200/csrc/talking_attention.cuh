// Arguments shared by the talking-heads attention kernels (talking_attention.cu has the mathematics).
#pragma once

#include "common.cuh"

namespace b200 {

constexpr int kTalkTileRows = 16;      // query rows per CTA of the prompt kernel

struct TalkArgs {
  const void* q;             // [rows, H, dk], row stride q_stride elements
  int64_t q_stride;
  const void* gate;          // [rows, H, dv] or null, row stride gate_stride
  int64_t gate_stride;
  const void* kc;            // [num_blocks, bs, Hkv, dk]
  const void* vc;            // [num_blocks, bs, Hkv, dv]
  void* out;                 // [rows, H, dv]
  const int32_t* bt;         // [n, bt_stride]
  int64_t bt_stride;
  int bs, bs_log2;           // bs_log2: -1 if bs is no power of two
  int64_t num_blocks;
  const int32_t* cu_q;       // [n + 1], or null: row i is the last token of sequence i
  const int32_t* cu_k;
  const int64_t* ctx_lens;   // [n] without cu_q; 0 = padding row
  int n;
  int64_t rows;
  int H, Hkv, dk, dv;
  float scale, cap;          // cap <= 0: no soft cap
  const float* r1;           // [H]
  const float* r2;           // [H]
  const float* talk;         // [H, H] out-head, in-head
  int window;                // <= 0: none
  const int32_t* plan;       // tile list of b200_prefill_plan for 16-row tiles, or null
  int plan_capacity;
  int max_q;                 // bound on rows per sequence
  const float* talk_host;    // talk on the host, or null
  const float* r1_host;      // r1, r2 on the host with talk_host
  const float* r2_host;
  const float* bias_table;   // [H, bias_len] r1 ln(1 + r2 distance), or null
  int bias_len;
  void* workspace;
  size_t workspace_bytes;
  int32_t* status;
};

// bf16 tensor-core paths; B200_ERR_UNSUPPORTED = sizes or alignments they do not take
int talking_prefill_mma_launch(const TalkArgs& a, cudaStream_t s);
int talking_decode_mma_launch(const TalkArgs& a, cudaStream_t s);
size_t talking_decode_workspace_bytes(int n, int H, int dv, int window);

}  // namespace b200
