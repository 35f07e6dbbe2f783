/*
 * b200llm.h — C ABI of the B200 (sm_100a) kernels behind the continuous-batching
 * prefill/decode step of the nano-vLLM-style engine in ZenoAFfectionate/LLM_from_Scratch.
 *
 * The reference engine has no native layer: its attention layer (the part that would call a
 * store_kvcache kernel, a varlen prefill attention and a paged decode attention) is missing from
 * the repository.  What the reference does define is the contract those kernels must honour —
 * the metadata tensors built by engine/model_runner.py (prepare_prefill :202-249, prepare_decode
 * :253-278), the KV pool layout of allocate_kv_cache (:162-190) and the padding conventions of
 * the CUDA-graph replay (:295-310).  Every entry point below cites the part of that contract it
 * implements.
 *
 * Conventions
 *   - every pointer is a BORROWED device pointer unless its name ends in _host; the library never
 *     allocates, frees or retains memory;
 *   - `stream` is a cudaStream_t passed as void*; a call only enqueues work on that stream and
 *     never synchronises the host, so every call can be captured in a CUDA graph;
 *   - metadata dtypes are exactly the reference's: slot_mapping and context_lens int64,
 *     block_tables and cu_seqlens int32; -1 is legal padding in slot_mapping and block_tables;
 *   - calls are reentrant and take no locks.  The only process-wide state is a few per-device caches (SM count,
 *     "shared-memory limit raised" flags, the address of the built-in scratch array) that are filled on first
 *     use without synchronisation: concurrent first calls from several host threads store identical values;
 *   - return value: 0 on success, a negative B200_ERR_* code for argument / launch errors that
 *     are detected on the host.  Faults detected on the device (a block id or slot outside the
 *     pool) never dereference the bad address: the access is skipped and a B200_ERR_* code is
 *     stored to `status` (a caller-owned device int32, may be NULL); read it with
 *     b200_read_status at the next host sync point;
 *   - dtype: B200_DTYPE_F32 or B200_DTYPE_BF16 is the element type of q/k/v/caches/outputs.
 *     Arithmetic is always accumulated in fp32.
 */
#ifndef B200LLM_H_
#define B200LLM_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define B200_ABI_VERSION 13

#define B200_DTYPE_F32 0
#define B200_DTYPE_BF16 1

#define B200_OK 0
#define B200_ERR_ARG (-1)          /* null pointer, negative size, inconsistent head counts */
#define B200_ERR_ALIGN (-2)        /* pointer or stride not aligned as the kernel requires   */
#define B200_ERR_UNSUPPORTED (-3)  /* shape / dtype outside what the kernels implement       */
#define B200_ERR_LAUNCH (-4)       /* the CUDA runtime refused the launch                    */
#define B200_ERR_WORKSPACE (-5)    /* workspace smaller than *_workspace_bytes asks for      */
#define B200_ERR_BOUNDS (-6)       /* device-side: block id or slot outside the pool         */
#define B200_ERR_NO_DEVICE (-7)    /* no usable CUDA device                                  */
#define B200_ERR_TOO_LARGE (-8)    /* scratch needed exceeds a fixed built-in capacity       */
#define B200_ERR_TIMEOUT (-9)      /* device-side: a bounded barrier wait gave up            */

int b200_abi_version(void);
const char* b200_strerror(int code);

/* Number of SMs of the current device (148 on B200); <0 on error. */
int b200_sm_count(void);

/* Copies the device status word to the host (synchronises `stream`) and clears it. */
int b200_read_status(int32_t* status, int32_t* status_host, void* stream);

/* ---------------------------------------------------------------------------------------------
 * XXH64 of a byte string with seed 0, and the chained block hash built on it.
 * Replaces BlockManager.compute_hash (engine/block_manager.py:45-57), which calls the third-party
 * xxhash package: hash = XXH64( [8-byte little-endian prefix hash, if prefix != -1] ||
 * int32-little-endian token ids ).  Host-only; no GPU work.
 * ------------------------------------------------------------------------------------------- */
uint64_t b200_xxh64(const void* data_host, size_t len, uint64_t seed);
uint64_t b200_block_hash(const int32_t* token_ids_host, int32_t num_tokens, uint64_t prefix_hash,
                         int32_t has_prefix);
/* The whole chain at once: out_hashes[i] for every full block i of the token list (prefix of block 0:
 * none, of block i: out_hashes[i-1]).  Returns the number of full blocks, or -1 on a bad argument. */
int64_t b200_block_hash_chain(const int32_t* token_ids_host, int64_t num_tokens, int32_t block_size,
                              uint64_t* out_hashes);

/* ---------------------------------------------------------------------------------------------
 * The KV-block pool on the host, natively: BlockManager (engine/block_manager.py:8-157) as a handle.  Blocks are
 * handed out oldest-free-first (the reference's FIFO deque, :60-78); full blocks are sealed with the chained
 * hash above and found again by later prompts (:85-114) after a token-by-token comparison; reference counts
 * start at 1 (the reference starts at 0 and so leaks unshared blocks, :23-26; this is the engine's corrected
 * default mode), a released block keeps its contents and can be revived, and a hit never covers a whole
 * prompt.  Host-only, no GPU work; a handle is not thread-safe.
 *   b200_pool_allocate    blocks for a new sequence (allocate, :85-114): writes ceil(num_tokens/block_size) block
 *                         ids, *num_cached_out = tokens covered by reused blocks; returns the number of
 *                         blocks, or B200_ERR_TOO_LARGE when the pool runs dry (state partly applied, as
 *                         the reference's IndexError would leave it)
 *   b200_pool_deallocate  releases a table, last block first (deallocate, :116-127)
 *   b200_pool_append      decode-time growth (append, :136-157): see the definition's comment
 *   b200_pool_open_block / b200_pool_seal_block  the two halves of append for several decode steps per
 *                         scheduling decision: open ahead, seal once the tokens are known
 *   b200_pool_lookup      the block a chained hash currently resolves to, or -1
 *   b200_pool_snapshot    free ids oldest first (returns their number), reference counts, sealed flags, hashes
 * ------------------------------------------------------------------------------------------- */
void* b200_pool_create(int64_t num_blocks, int32_t block_size);
void b200_pool_destroy(void* pool);
int64_t b200_pool_num_free(const void* pool);
int64_t b200_pool_allocate(void* pool, const int32_t* token_ids_host, int64_t num_tokens, int32_t* table_out_host,
                           int64_t* num_cached_out_host);
int b200_pool_deallocate(void* pool, const int32_t* table_host, int64_t num_blocks);
int64_t b200_pool_append(void* pool, int32_t last_block, int32_t prev_block, int64_t num_tokens,
                         const int32_t* last_block_tokens_host);
int64_t b200_pool_open_block(void* pool);
int b200_pool_seal_block(void* pool, int32_t block, int32_t prev_block, const int32_t* block_tokens_host);
int64_t b200_pool_lookup(const void* pool, uint64_t hash);
int64_t b200_pool_snapshot(const void* pool, int32_t* free_order_host, int32_t* ref_counts_host,
                           uint8_t* sealed_host, uint64_t* hashes_host);

/* ---------------------------------------------------------------------------------------------
 * Step metadata on the host, natively (ModelRunner.prepare_prefill / prepare_decode, engine/model_runner.py:
 * 202-278), written straight into caller-owned (pinned) arrays.  Block tables arrive as one flat int32 array
 * with offsets: sequence i owns tables[table_offsets[i] : table_offsets[i + 1]].
 *   b200_prepare_prefill  the non-cached suffix of every sequence: cu_seqlens_q / cu_seqlens_k int32 [n + 1],
 *                         positions int64 [T] (num_cached + j for packed token j), slot_mapping int64 [T],
 *                         max_seqlens[0..1] = longest q / k; returns T (<= capacity) or a negative code
 *   b200_prepare_decode   one token per sequence: context_lens, slot_mapping int64 [n], block_tables int32
 *                         [n, width] padded with -1
 * ------------------------------------------------------------------------------------------- */
int64_t b200_prepare_prefill(int32_t num_seqs, const int64_t* num_tokens_host, const int64_t* num_cached_host,
                             const int64_t* table_offsets_host, const int32_t* tables_host, int32_t block_size,
                             int32_t* cu_seqlens_q_host, int32_t* cu_seqlens_k_host, int64_t* positions_host,
                             int64_t* slot_mapping_host, int64_t capacity, int32_t* max_seqlens_host);
int b200_prepare_decode(int32_t num_seqs, const int64_t* num_tokens_host, const int64_t* table_offsets_host,
                        const int32_t* tables_host, int32_t block_size, int64_t* context_lens_host,
                        int64_t* slot_mapping_host, int32_t* block_tables_host, int64_t width);

/* ---------------------------------------------------------------------------------------------
 * store_kvcache: k_cache[slot_mapping[t], :, :] = k[t, :, :] (same for v); slot < 0 is skipped.
 * Contract: engine/model_runner.py:184-190 (pool [num_blocks, block_size, Hkv, D] per layer, so a
 * slot is one row of [num_slots, Hkv*D]), :226-230 (prefill slots), :261 (decode slot) and
 * :300-301 (-1 padding under graph replay).
 *   k, v            [num_tokens, Hkv, D]; rows Hkv*D contiguous, token stride given in ELEMENTS
 *                   (k/v may be column slices of a fused qkv projection)
 *   k_cache,v_cache [num_slots, Hkv, D] contiguous
 *   v and v_cache may both be NULL for a single pool (the MLA latent cache: Hkv = 1,
 *   D = kv_lora_rank + rope_dim)
 * ------------------------------------------------------------------------------------------- */
int b200_store_kvcache(const void* k, const void* v, int64_t k_token_stride,
                       int64_t v_token_stride, void* k_cache, void* v_cache,
                       const int64_t* slot_mapping, int32_t num_tokens, int32_t num_kv_heads,
                       int32_t head_dim, int64_t num_slots, int32_t dtype, int32_t* status,
                       void* stream);

/* ---------------------------------------------------------------------------------------------
 * Paged GQA decode attention: one query token per sequence attends to its whole context through
 * block_tables.  Arithmetic = GroupedQueryAttention.forward cache branch
 * (model/attention/GQA.py:105-130) with the dense cache replaced by the paged pool; metadata =
 * prepare_decode (engine/model_runner.py:253-278).
 *   q, out        [batch, Hq, D] contiguous
 *   k_cache       [num_blocks, block_size, Hkv, D]
 *   block_tables  [batch, bt_stride] int32, entries beyond ceil(context_len/block_size) are
 *                 never read (-1 or stale values are fine)
 *   context_lens  [batch] int64, includes the token being decoded; <= 0 writes a zero row
 *   workspace     b200_paged_decode_gqa_workspace_bytes(...) bytes, 256-byte aligned; holds the arrival
 *                 counters and partial results of contexts split across thread blocks.  Its first
 *                 B200_DECODE_COUNTER_BYTES must be zero when the buffer is first used (one cudaMemset after
 *                 allocating it); every call leaves them zero again, whatever the shapes of successive calls.
 *                 The rest needs no initialisation.  Two calls that overlap on the GPU need two workspaces.
 * ------------------------------------------------------------------------------------------- */
#define B200_DECODE_COUNTER_BYTES ((size_t)256 << 10)
size_t b200_paged_decode_gqa_workspace_bytes(int32_t batch, int32_t num_q_heads,
                                             int32_t num_kv_heads, int32_t head_dim,
                                             int32_t dtype);
int b200_paged_decode_gqa(const void* q, const void* k_cache, const void* v_cache, void* out,
                          const int32_t* block_tables, int64_t bt_stride,
                          const int64_t* context_lens, int32_t batch, int32_t num_q_heads,
                          int32_t num_kv_heads, int32_t head_dim, int32_t block_size,
                          int64_t num_blocks, float scale, void* workspace, size_t workspace_bytes,
                          int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Paged GQA decode for callers that cannot allocate device memory (no counterpart in the
 * reference, whose engine allocates freely through torch).  Same arguments and results as
 * b200_paged_decode_gqa minus the workspace: the split-context scratch is a fixed
 * B200_STATIC_SCRATCH_BYTES (8 MiB) device array inside the library, held by every GPU that loads
 * the library until the process exits.  It is meant for hosts that gave all
 * device memory to the KV pool, or that may not call an allocator on the decode path.
 *   - calls no cudaMalloc/cudaFree or any allocating routine;
 *   - returns B200_ERR_TOO_LARGE when the call would take the split-context kernel (bf16, block_size 16,
 *     head_dim 32/64/128, 16-byte aligned q and caches) and b200_paged_decode_gqa_workspace_bytes(...) for
 *     the shape exceeds the capacity (nothing is launched); shapes served by the general kernel need no
 *     scratch and are never refused;
 *   - the first call on each device looks up the array's device address (a host-side symbol query,
 *     made with that device current); make that first call before starting any stream capture;
 *   - all calls share the array: calls that overlap on the GPU (two streams, two threads) race on
 *     it.  Nothing in it has to be cleared between calls (the counters at its head start at zero when the
 *     library is loaded and every call returns them to zero).
 * ------------------------------------------------------------------------------------------- */
#define B200_STATIC_SCRATCH_BYTES ((size_t)8 << 20)
int b200_paged_decode_gqa_static(const void* q, const void* k_cache, const void* v_cache,
                                 void* out, const int32_t* block_tables, int64_t bt_stride,
                                 const int64_t* context_lens, int32_t batch, int32_t num_q_heads,
                                 int32_t num_kv_heads, int32_t head_dim, int32_t block_size,
                                 int64_t num_blocks, float scale, int32_t dtype, int32_t* status,
                                 void* stream);

/* ---------------------------------------------------------------------------------------------
 * Ragged (varlen) causal prefill attention over sequences packed with cu_seqlens.
 * Arithmetic = scaled_dot_product_attention (model/attention/utils.py:51-63) per sequence with
 * the causal mask of TransformerLM.forward (model/transformer.py:174-176), bottom-right aligned
 * when seqlen_k > seqlen_q (GQA.py:108-113), KV heads shared as GQA.py:118-125; metadata =
 * prepare_prefill (engine/model_runner.py:202-249).
 *   q   [total_q, Hq, Dqk]   token stride q_token_stride (elements), heads contiguous
 *   k   [total_k, Hkv, Dqk], v [total_k, Hkv, Dv]: the new tokens' keys/values when
 *       block_tables == NULL (then cu_seqlens_k must equal cu_seqlens_q);
 *   when block_tables != NULL (some prefix is cached, model_runner.py:231-237) keys/values are
 *       read from k_cache/v_cache through block_tables [num_seqs, bt_stride] and k/v are ignored
 *       (the caller has already stored the new tokens with b200_store_kvcache);
 *   out [total_q, Hq, Dv] contiguous.
 *   total_q_tokens / total_k_tokens are the row counts of q and of k/v (>= cu_seqlens[num_seqs],
 *   which the host knows from its tensors): they bound the TMA tensor maps built over q/k/v.
 *   plan (may be NULL): a tile list written by b200_prefill_plan for the same cu_seqlens_q, with its
 *   tile_rows and capacity.  With a plan the tiled kernels launch one CTA per listed tile (longest
 *   first) instead of num_seqs x ceil(max_seqlen_q / tile) CTAs, and neither num_seqs nor max_seqlen_q
 *   shapes the grid any more, so a step with fixed buffer sizes can be captured in a CUDA graph:
 *   pass num_seqs = the capacity of cu_seqlens (unused trailing sequences have length 0).
 *   A plan whose tile_rows does not match the kernel chosen for the shape is ignored.
 *   slot_mapping (may be NULL): int64, one slot per new token (the rows of k / v; -1 = skip), as prepare_prefill
 *   builds it (model_runner.py:226-230).  When given, the call also performs the step's store_kvcache:
 *   k_cache[slot] = k row, v_cache[slot] = v row for the pool [num_blocks, block_size, Hkv, D] (k, v, k_cache,
 *   v_cache, block_size and num_blocks are then required, with or without block_tables, and head_dim_qk must
 *   equal head_dim_v).  The scatter is enqueued ahead of the attention grid inside this call, so keys read
 *   through block_tables include the new tokens.
 * ------------------------------------------------------------------------------------------- */
int b200_prefill_varlen(const void* q, const void* k, const void* v, void* out,
                        int64_t q_token_stride, int64_t k_token_stride, int64_t v_token_stride,
                        int64_t total_q_tokens, int64_t total_k_tokens,
                        const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                        int32_t num_seqs, int32_t max_seqlen_q, int32_t max_seqlen_k,
                        int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                        int32_t head_dim_v, float scale, const void* k_cache, const void* v_cache,
                        const int32_t* block_tables, int64_t bt_stride, int32_t block_size,
                        int64_t num_blocks, const int64_t* slot_mapping, const int32_t* plan,
                        int32_t plan_tile_rows, int32_t plan_capacity, int32_t dtype, int32_t* status,
                        void* stream);

/* The same attention for keys stored in two parts, as the expanded form of multi-head latent attention
 * has them (model/attention/MLA.py:93-95,131: k = [k_nope of the head | k_rope shared by all heads]):
 *   k_head [total_k, H, head_dim_qk - tail_dim]  per-head columns, token stride k_head_token_stride
 *   k_tail [total_k, tail_dim]                   last tail_dim columns of every head's key
 *   q      [total_q, H, head_dim_qk], v [total_k, H, head_dim_v], out [total_q, H, head_dim_v]
 * so the rotary part is never copied into every head.  Keys/values are packed (no paged prefix);
 * total_q_tokens / total_k_tokens are the row counts of q and of k_head / k_tail / v, as above.
 * bf16, (head_dim_qk, tail_dim, head_dim_v) = (192, 64, 128), all parts 16-byte aligned; anything else
 * returns B200_ERR_UNSUPPORTED (the caller then expands the keys and uses b200_prefill_varlen).  plan: as above, for the
 * tile_rows of b200_prefill_tile_rows(head_dim_qk, head_dim_v, H, H, dtype). */
int b200_prefill_varlen_shared_tail(const void* q, const void* k_head, const void* k_tail, const void* v,
                                    void* out, int64_t q_token_stride, int64_t k_head_token_stride,
                                    int64_t k_tail_token_stride, int64_t v_token_stride,
                                    int64_t total_q_tokens, int64_t total_k_tokens,
                                    const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                    int32_t num_seqs, int32_t max_seqlen_q, int32_t num_heads,
                                    int32_t head_dim_qk, int32_t tail_dim, int32_t head_dim_v, float scale,
                                    const int32_t* plan, int32_t plan_tile_rows, int32_t plan_capacity,
                                    int32_t dtype, int32_t* status, void* stream);

/* Tile list for b200_prefill_varlen, computed on the device from cu_seqlens_q (one small launch per
 * step; all layers of the step reuse it).
 *   b200_prefill_tile_rows: query rows per tile of the kernel that serves this shape with packed keys
 *     (256 or 128 tcgen05: head dims 128 / 192+128, and head_dim 64 with query heads in groups of four;
 *     64 mma.sync), or 0 when only the general kernel applies (no plan then).
 *   b200_prefill_plan_bytes: size of `plan` for up to total_q_tokens rows in up to num_seqs sequences;
 *     its capacity in tiles is bytes / 4 - 4.
 *   b200_prefill_plan: max_seqlen_q is a host-side upper bound of the longest sequence
 *     (more than 4096 tiles in one sequence: B200_ERR_UNSUPPORTED).  Layout: int32 header
 *     {tiles, tile_rows, capacity, 0}, then (sequence << 16 | tile) per tile, highest tiles first. */
int32_t b200_prefill_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                               int32_t head_dim_v, int32_t dtype);
size_t b200_prefill_plan_bytes(int64_t total_q_tokens, int32_t num_seqs, int32_t tile_rows);
int b200_prefill_plan(const int32_t* cu_seqlens_q, int32_t num_seqs, int32_t max_seqlen_q,
                      int32_t tile_rows, int32_t* plan, size_t plan_bytes, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * MLA latent-cache decode (absorbed form).  Arithmetic = MultiHeadLatentAttention.forward cache
 * branch (model/attention/MLA.py:153-178) between the two weight einsums:
 *   score = (q_abs . c^T + q_rope . pe^T) * scale ; P = softmax(score) ; out_latent = P . c
 * with c/pe read from a paged latent pool whose rows are [kv_lora_rank | rope_dim].
 *   q_abs [batch, H, r], q_rope [batch, H, dr], out_latent [batch, H, r] contiguous
 *   latent_cache [num_blocks, block_size, r + dr]
 * ------------------------------------------------------------------------------------------- */
size_t b200_mla_decode_workspace_bytes(int32_t batch, int32_t num_heads, int32_t kv_lora_rank,
                                       int32_t rope_dim, int32_t dtype);
int b200_mla_decode(const void* q_abs, const void* q_rope, const void* latent_cache,
                    void* out_latent, const int32_t* block_tables, int64_t bt_stride,
                    const int64_t* context_lens, int32_t batch, int32_t num_heads,
                    int32_t kv_lora_rank, int32_t rope_dim, int32_t block_size,
                    int64_t num_blocks, float scale, void* workspace, size_t workspace_bytes,
                    int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Residual-stream RMSNorm with the reference's optional fused residual add (model/utils.py:54-67):
 *   xf = float(x) [+ float(residual)];  y = (weight * xf * rsqrt(mean(xf^2) + eps)) in x's dtype;
 *   residual_out = xf in x's dtype (may be NULL).  x, y, residual_out: [num_rows, dim] contiguous in
 *   `dtype`; residual (may be NULL) in `residual_dtype`; weight fp32 [dim].
 * ------------------------------------------------------------------------------------------- */
int b200_add_rmsnorm(const void* x, const void* residual, const float* weight, void* y,
                     void* residual_out, int64_t num_rows, int32_t dim, float eps, int32_t dtype,
                     int32_t residual_dtype, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Everything GroupedQueryAttention.forward does between its projections and the attention call
 * (model/attention/GQA.py:81-102), plus the store_kvcache scatter, in one pass over the fused
 * projection output qkv [num_tokens, >= (Hq + 2 Hkv) * D] (token stride in elements):
 *   q, k: RMSNorm over the whole projected vector (eps as given: the reference's layers have eps=None,
 *   which torch evaluates in fp32 with the fp32 machine epsilon when the weight is fp32), rounded to the
 *   dtype, then half-split RoPE (model/attention/utils.py:34-45) in fp32 at positions[t] using rope_table [rope_positions, D] = cat(cos, sin), rounded to the dtype;
 *   q_out [num_tokens, Hq, D], k_out [num_tokens, Hkv, D];
 *   if k_cache != NULL: k_cache[slot] = k_out row, v_cache[slot] = raw v row, slot < 0 skipped.
 * ------------------------------------------------------------------------------------------- */
int b200_qk_norm_rope_store(const void* qkv, int64_t qkv_token_stride, const float* q_norm_weight,
                            const float* k_norm_weight, const float* rope_table,
                            int64_t rope_positions, const int64_t* positions, void* q_out, void* k_out,
                            void* k_cache, void* v_cache, const int64_t* slot_mapping,
                            int64_t num_slots, int64_t num_tokens, int32_t num_q_heads,
                            int32_t num_kv_heads, int32_t head_dim, float eps, int32_t dtype,
                            int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Everything MultiHeadLatentAttention.forward does between its projections and the attention
 * (model/attention/MLA.py:114-131 and the cache write of :137-138), one pass per token:
 *   q_up    [num_tokens, >= H*head_dim + H*rope_dim] (row stride in elements): the fused q up-projection,
 *           q_nope of all heads followed by q_rope of all heads;
 *   kv_down [num_tokens, >= kv_lora_rank + rope_dim]: the kv down-projection followed by k_rope.
 *   q_out    [num_tokens, H, head_dim + rope_dim] = [ q_nope | RoPE(q_rope) ]
 *   rows_out [num_tokens, kv_lora_rank + rope_dim] = [ RMSNorm(c) * kv_norm_weight | RoPE(k_rope) ]
 *            (may be NULL); the same row is written to latent_cache[slot_mapping[t]] when
 *            latent_cache != NULL (slot < 0 skipped).
 * RoPE is half-split, fp32, and reads cos from rope_table[pos, 0 : rope_dim/2] and "sin" from
 * rope_table[pos, rope_dim/2 : rope_dim]: the reference slices a table built for head_dim to its first
 * rope_dim columns (model/attention/utils.py:38), which this reproduces.  bf16 only.
 * ------------------------------------------------------------------------------------------- */
int b200_mla_prologue(const void* q_up, int64_t q_up_stride, const void* kv_down, int64_t kv_down_stride,
                      const float* kv_norm_weight, const float* rope_table, int64_t rope_width,
                      int64_t rope_positions, const int64_t* positions, void* q_out, void* rows_out,
                      void* latent_cache, const int64_t* slot_mapping, int64_t num_slots,
                      int64_t num_tokens, int32_t num_heads, int32_t head_dim, int32_t rope_dim,
                      int32_t kv_lora_rank, float eps, int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * MoE routing for inference (Gate.forward, model/architecture/moe.py:45-90, and the grouping by
 * expert that MOE.moe_infer does with argsort + bincount on the host, moe.py:297-307), on the device.
 *   gate_logits [num_tokens, num_experts] in `dtype` (= x @ gate_weight^T), expert_bias fp32.
 *   scores = sigmoid(logits); top_k experts by logits + bias (ties to the lower index); weights =
 *   selected scores / (their sum + 1e-10) when top_k > 1; all rounded as the dtype would.
 * Outputs, rows ordered by (expert, token):
 *   sorted_token / sorted_expert int32 [num_tokens*top_k], sorted_weight `dtype` [num_tokens*top_k],
 *   expert_offsets int32 [num_experts] (exclusive end of every expert's rows),
 *   slot_to_row int32 [num_tokens, top_k]: row of token t's j-th expert in ascending expert order.
 * identity_tail != 0: sorted_token has num_tokens*top_k + num_tokens entries and the last num_tokens are
 *   0, 1, 2, ...: one gather then also yields the rows of a shared expert (see b200_moe_grouped_gemm).
 * One launch for num_tokens <= 256, two (count, scatter) above; `workspace` of
 * b200_moe_route_workspace_bytes() bytes (0 for num_tokens <= 256) holds the per-CTA counts.
 * Limits: num_experts <= 64, top_k <= 8, num_tokens <= 65536 (else B200_ERR_UNSUPPORTED).
 * ------------------------------------------------------------------------------------------- */
size_t b200_moe_route_workspace_bytes(int32_t num_tokens, int32_t num_experts);
int b200_moe_route(const void* gate_logits, const float* expert_bias, int32_t num_tokens,
                   int32_t num_experts, int32_t top_k, int32_t* sorted_token, int32_t* sorted_expert,
                   void* sorted_weight, int32_t* expert_offsets, int32_t* slot_to_row,
                   int32_t identity_tail, void* workspace, size_t workspace_bytes, int32_t dtype,
                   void* stream);

/* The gate projection, the routing above and (optionally) the gather of the routed rows in ONE launch, for
 * batches of at most 256 tokens (decode): gate_logits = bf16(x . gate_weight^T) (Gate.forward, moe.py:49-52),
 * then exactly b200_moe_route.  x [num_tokens, d_model] bf16 contiguous, gate_weight [num_experts, d_model] bf16.
 * gathered (may be NULL): [num_tokens*top_k (+ num_tokens with identity_tail), d_model], row i = x[sorted_token[i]]
 * (the index_select that feeds b200_moe_grouped_gemm); one thread block copies the rows, so pass it for small
 * batches only.  workspace: b200_moe_gate_route_workspace_bytes() bytes, 256-byte aligned, zero when first
 * used (its first word is a ticket counter that every call returns to zero).  More than 256 tokens, another
 * dtype, d_model % 8 != 0 or a gate matrix above 160 KiB: B200_ERR_UNSUPPORTED (use a GEMM and b200_moe_route). */
size_t b200_moe_gate_route_workspace_bytes(void);
int b200_moe_gate_route(const void* x, const void* gate_weight, const float* expert_bias, int32_t num_tokens,
                        int32_t num_experts, int32_t top_k, int32_t d_model, int32_t* sorted_token,
                        int32_t* sorted_expert, void* sorted_weight, int32_t* expert_offsets,
                        int32_t* slot_to_row, int32_t identity_tail, void* gathered, void* workspace,
                        size_t workspace_bytes, int32_t dtype, void* stream);

/* ---------------------------------------------------------------------------------------------
 * SwiGLU of fused up-projection rows (model/architecture/mlp.py:61-67: w2(silu(w1 x) * w3 x)):
 *   h [num_rows, 2*d_ff] = [w1 x | w3 x];  act [num_rows, d_ff] = silu(h1 + b1) * (h3 + b3).
 * `bias` (may be NULL: already added by the GEMM) is [experts, 2*d_ff]; row r uses the bias row
 * row_expert[r] (row 0 when row_expert is NULL).  Bias add, silu and product are each rounded to the
 * dtype, like the tensor-op sequence they replace.
 * ------------------------------------------------------------------------------------------- */
int b200_swiglu(const void* h, const void* bias, const int32_t* row_expert, void* act, int64_t num_rows,
                int32_t d_ff, int32_t dtype, void* stream);

/* ---------------------------------------------------------------------------------------------
 * MoE combine (MOE.moe_infer, moe.py:312-339, and the shared expert, moe.py:272-273):
 *   out[t] = sum_j round(round(expert_out[row] + bias[row_expert[row]]) * row_weight[row]),
 *   row = slot_to_row[t, j], j ascending (= ascending expert id), every partial sum rounded to the
 *   dtype as the reference's scatter_add_ in the activation dtype does; then + shared[t] if given.
 * expert_out [num_tokens*top_k, d_model] in grouped (sorted) row order; bias [experts, d_model] or NULL.
 * ------------------------------------------------------------------------------------------- */
int b200_moe_combine(const void* expert_out, const void* bias, const int32_t* row_expert,
                     const void* row_weight, const int32_t* slot_to_row, const void* shared, void* out,
                     int64_t num_tokens, int32_t top_k, int32_t d_model, int32_t dtype, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Grouped GEMM over rows grouped by expert (the per-expert loop of MOE.moe_infer, moe.py:299-339),
 * bf16, fp32 accumulation on the tensor cores.  Expert e owns rows [offsets[e-1], offsets[e]) of
 * x [num_rows, k_dim] (expert_offsets as b200_moe_route writes them; read on the device).
 *   mode 0: out [num_rows, n_out] = x . W_e^T (+ bias[e] if given), w [experts, n_out, k_dim].
 *   mode 1: out [num_rows, n_out] = silu(x . W1_e^T + b1) * (x . W3_e^T + b3), n_out = d_ff,
 *           w [experts, 2*d_ff, k_dim] = rows of w1 then rows of w3, bias [experts, 2*d_ff] or NULL
 *           (mlp.py:61-67); GEMM result, bias add, silu and product are each rounded to bf16.
 * dense_rows > 0: the last dense_rows of the num_rows rows are not grouped: they all use weight set
 *   number num_experts (w and bias then hold num_experts + 1 sets) — a shared expert applied to every token
 *   (moe.py:272-273) computed by the same launch, in chunks that cost a CTA what an expert's rows cost.
 * mode | B200_MOE_GEMM_EARLY_LAUNCH: the launch is a programmatic dependent of the kernel before it in
 *   the stream: the prologue and the first ring of weight tiles overlap that kernel's tail, and only the
 *   reads of x wait for it.  The caller asserts that w, bias and expert_offsets were complete before
 *   that kernel started (they come from two or more launches back, as in route -> gather -> up -> down).
 * Requires k_dim % 8 == 0 and 16-byte aligned x, w (B200_ERR_ALIGN).  A wait that runs out inside
 * the kernel sets *status to B200_ERR_TIMEOUT.
 * ------------------------------------------------------------------------------------------- */
#define B200_MOE_GEMM_EARLY_LAUNCH 0x100
int b200_moe_grouped_gemm(const void* x, const void* w, const void* bias, void* out,
                          const int32_t* expert_offsets, int64_t num_rows, int32_t num_experts,
                          int32_t dense_rows, int32_t n_out, int32_t k_dim, int32_t mode, int32_t dtype,
                          int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Decode metadata of the next step, computed on the device from the step that just ran, so that several
 * decode steps can be launched back to back (host counterpart: ModelRunner.prepare_decode,
 * engine/model_runner.py:253-278).  For every row i < num_seqs:
 *   input_ids[i] = sampled[i];  context_lens[i] += 1;
 *   slot_mapping[i] = block_tables[i, (len-1)/block_size] * block_size + (len-1) % block_size  (len = new length)
 *   history[i] = sampled[i] when history != NULL (the host reads all steps' tokens at the end).
 * block_tables int32 [num_seqs, bt_stride] must already list the block the new token falls into; a table
 * that does not sets the slot to -1 and reports B200_ERR_BOUNDS in *status.
 * ------------------------------------------------------------------------------------------- */
int b200_decode_advance(const int64_t* sampled, int64_t* input_ids, int64_t* context_lens,
                        int64_t* slot_mapping, const int32_t* block_tables, int64_t bt_stride,
                        int32_t block_size, int64_t num_blocks, int32_t num_seqs, int64_t* history,
                        int32_t* status, void* stream);

/* Device-resident block tables: writes `count` (row, column, block id) int32 triples into
 * block_tables [rows, bt_stride], so that a decode step uploads only the table entries that changed since
 * the previous step (the reference rebuilds and ships the whole table, engine/model_runner.py:263-268).
 * A triple outside the table is skipped and reported as B200_ERR_BOUNDS in *status. */
int b200_block_table_patch(const int32_t* patches, int32_t count, int32_t* block_tables, int64_t bt_stride,
                           int32_t rows, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Token sampling (Sampler.forward, utils/sampler.py:35-52; greedy argmax of generate.py:62), one launch.
 *   logits [num_rows, >= vocab_size] (row stride in elements) in `dtype`; temperatures fp32 [num_rows] or
 *   NULL (= all greedy).  Row r with temperature T > 0: a draw from softmax(logits[r] / T) as the
 *   exponential race argmax_i (logits_i / T - log E_i), E_i ~ Exp(1) clamped at 1e-10 like the reference;
 *   T <= 0: argmax of the logits, lowest index among equal maxima.  out_tokens int64 [num_rows].
 *   The uniforms are a counter-based function of (seed, offset, row, element): pass a fresh `offset` per
 *   step.  The stream differs from torch's, so only the distribution matches the reference.
 * ------------------------------------------------------------------------------------------- */
int b200_sample(const void* logits, int64_t row_stride, const float* temperatures, int64_t num_rows,
                int32_t vocab_size, uint64_t seed, uint64_t offset, int64_t* out_tokens, int32_t dtype,
                void* stream);

/* ---------------------------------------------------------------------------------------------
 * Greedy head in two launches: the lm_head projection (TransformerLM.lm_head, model/transformer.py:160,183)
 * fused with the greedy argmax of generate.py:62 / the T = 0 rows of the sampler:
 *   tokens[r] = argmax_v bf16( hidden[r] . W[v] + bias[v] ), lowest v among equal maxima,
 * i.e. what argmax over the bf16 logits of a biased linear layer returns, without writing the logits.
 *   hidden [num_rows, k_dim] bf16 contiguous, w [vocab_size, k_dim] bf16, bias [vocab_size] bf16 or NULL,
 *   tokens int64 [num_rows]; workspace of b200_lm_head_argmax_workspace_bytes() bytes, 256-byte aligned
 *   (per-tile maxima; nothing survives the call).  tcgen05 kernel that streams W once; bf16 only, k_dim % 8 == 0.
 * ------------------------------------------------------------------------------------------- */
size_t b200_lm_head_argmax_workspace_bytes(int32_t num_rows, int32_t vocab_size);
int b200_lm_head_argmax(const void* hidden, const void* w, const void* bias, int64_t* tokens, int32_t num_rows,
                        int32_t vocab_size, int32_t k_dim, void* workspace, size_t workspace_bytes,
                        int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Mechanisms of decoders with hyper-connected residual streams, talking-heads attention and a gated linear
 * recurrence (the Nabalix family; the reference has no counterpart).  All constants are parameters.
 * ------------------------------------------------------------------------------------------- */

/* store_kvcache for a pool whose key and value rows differ in width: k_cache [num_slots, k_width],
 * v_cache [num_slots, v_width]; strides in elements, slots < 0 are skipped. */
int b200_store_kv_rows(const void* k, const void* v, int64_t k_token_stride, int64_t v_token_stride, void* k_cache,
                       void* v_cache, const int64_t* slot_mapping, int32_t num_tokens, int32_t k_width,
                       int32_t v_width, int64_t num_slots, int32_t dtype, int32_t* status, void* stream);

/* One sublayer boundary of a decoder with `streams` (1..8) fp32 residual streams x [rows, streams, dim], in place:
 *   y     = y0, or (rms(y0) join_w0 + rms(y1) join_w1) / 2 with y1 (eps join_eps); times layer_scale [dim] if given
 *   x'[t] = sum_s mix[s, t] x[s] + out_w[t] y          (mix [streams, streams] from-to; y0 == NULL: x' = x)
 *   u     = sum_t in_w[t] x'[t]                        (in_w == NULL: the plain sum)
 *   h     = u / sqrt(mean(u^2) + eps) * (norm_w + (norm_plus_one ? 1 : 0))     in `dtype`; h == NULL: not formed
 * With `embed` [vocab, dim] (dtype) and tokens int64 [rows] every stream starts as the token's row (no update).
 * y0, y1 [rows, dim] in dtype; all other vectors fp32.  A token id outside the table reads row 0 and reports
 * B200_ERR_BOUNDS. */
int b200_stream_update(float* x, const int64_t* tokens, const void* embed, int64_t vocab, const void* y0, const void* y1,
                       const float* join_w0, const float* join_w1, float join_eps, const float* layer_scale,
                       const float* mix, const float* out_w, const float* in_w, const float* norm_w,
                       int32_t norm_plus_one, float eps, void* h, int64_t rows, int32_t streams, int32_t dim,
                       int32_t dtype, int32_t* status, void* stream);

/* act [rows, d_ff] = g sigmoid(slope g) (u + 1) for h [rows, 2 d_ff] = [gate | up], g = min(gate, limit),
 * u = clamp(up, -limit, limit); fp32 arithmetic, one rounding. */
int b200_clamped_glu(const void* h, void* act, int64_t rows, int32_t d_ff, float limit, float slope, int32_t dtype,
                     void* stream);

/* Causal attention over a paged pool with heads mixed before the softmax; for a query at position i
 *   s[g, j] = softcap tanh(scale q[g].k[j] / softcap) - r1[g] ln(1 + r2[g] (i - j))   (softcap <= 0: no cap)
 *   m[h, j] = sum_g talk[h, g] s[g, j],  softmax over 0 <= i - j < window (window <= 0: all earlier keys),
 *   out[h]  = sum_j softmax(m[h])_j v[j] * sigmoid(gate[h])                            (gate == NULL: no gate)
 * Query head h reads key / value head h / (num_heads / num_kv_heads).  q [rows, num_heads * dim_k], gate
 * [rows, num_heads * dim_v] with free row strides; out [rows, num_heads, dim_v]; caches [num_blocks, block_size,
 * num_kv_heads, dim].  The rows of sequence s are cu_seqlens_q[s] .. cu_seqlens_q[s+1]-1, its context (which the
 * pool already holds, the new rows included) is cu_seqlens_k[s+1]-cu_seqlens_k[s] long; with cu_seqlens_q ==
 * NULL row i is the last token of sequence i and context_lens[i] its length (0: padding row, nothing written).
 * Rows beyond the last sequence are padding.  max_seqlen_q: host bound on rows per sequence.
 * r1, r2 [num_heads] and talk [num_heads, num_heads] fp32 (device); bias_table [num_heads, bias_len] fp32
 * or NULL: r1 ln(1 + r2 distance) for distances 0 .. bias_len - 1, bias_len >= window if given; consts_host: talk,
 * r1, r2 one after the other on the host (NULL: the general kernel runs).  plan: tile list of b200_prefill_plan for
 * B200_TALKING_TILE_ROWS rows per tile, or NULL.  Workspace: b200_talking_attention_workspace_bytes(). */
#define B200_TALKING_TILE_ROWS 16
size_t b200_talking_attention_workspace_bytes(int32_t num_seqs, int32_t num_heads, int32_t dim_v, int32_t window,
                                              int32_t decode, int32_t dtype);
int b200_talking_attention(const void* q, int64_t q_stride, const void* gate, int64_t gate_stride, const void* k_cache,
                           const void* v_cache, void* out, const int32_t* block_tables, int64_t bt_stride,
                           int32_t block_size, int64_t num_blocks, const int32_t* cu_seqlens_q,
                           const int32_t* cu_seqlens_k, const int64_t* context_lens, int32_t num_seqs, int64_t rows,
                           int32_t max_seqlen_q, int32_t num_heads, int32_t num_kv_heads, int32_t dim_k, int32_t dim_v,
                           float scale, float softcap, const float* r1, const float* r2, const float* talk,
                           const float* consts_host, const float* bias_table, int32_t bias_len, int32_t window,
                           const int32_t* plan, int32_t plan_tile_rows, int32_t plan_capacity, void* workspace,
                           size_t workspace_bytes, int32_t dtype, int32_t* status, void* stream);

/* Gated linear recurrence (HGRN2) over per-sequence states: per head
 *   q = silu(q_in), f = lower + (1 - lower) sigmoid(f_in + f_bias), S <- diag(f) S + (1 - f) v^T, o = S^T q,
 *   out = o / sqrt(mean(o^2) + eps) * norm_w
 * q, f [tokens, heads * dim_k], v [tokens, heads * dim_v] with one token stride (views of one projection);
 * f_bias, lower [heads, dim_k], norm_w [dim_v] fp32; state fp32 [num_slots, heads, dim_k, dim_v], slot of
 * sequence s = state_slots[s] (< 0: skipped).  Sequence ranges as in b200_talking_attention; a sequence whose
 * first token of the call is at position 0 starts from the zero state.  out [tokens, heads, dim_v] in dtype.
 * max_seqlen_q, total_tokens: host bounds (workspace: b200_gated_recurrence_workspace_bytes()). */
size_t b200_gated_recurrence_workspace_bytes(int32_t num_seqs, int64_t total_tokens, int32_t max_seqlen_q,
                                             int32_t num_heads, int32_t dim_k, int32_t dim_v);
int b200_gated_recurrence(const void* q, const void* f, const void* v, int64_t token_stride, const float* f_bias,
                          const float* lower, const float* norm_w, float eps, float* state, int64_t num_slots,
                          const int64_t* state_slots, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                          const int64_t* context_lens, int32_t num_seqs, int64_t total_tokens, int32_t max_seqlen_q,
                          int32_t num_heads, int32_t dim_k, int32_t dim_v, void* out, void* workspace,
                          size_t workspace_bytes, int32_t dtype, int32_t* status, void* stream);

/* b200_prefill_varlen with an attention sink: exp(sink[h]) (fp32 [num_q_heads], device; NULL: none) joins the softmax
 * denominator of query head h, without a key, a value or the scale. */
int b200_prefill_varlen_sink(const void* q, const void* k, const void* v, void* out, int64_t q_token_stride,
                             int64_t k_token_stride, int64_t v_token_stride, int64_t total_q_tokens,
                             int64_t total_k_tokens, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                             int32_t num_seqs, int32_t max_seqlen_q, int32_t max_seqlen_k, int32_t num_q_heads,
                             int32_t num_kv_heads, int32_t head_dim_qk, int32_t head_dim_v, float scale,
                             const void* k_cache, const void* v_cache, const int32_t* block_tables, int64_t bt_stride,
                             int32_t block_size, int64_t num_blocks, const int64_t* slot_mapping, const int32_t* plan,
                             int32_t plan_tile_rows, int32_t plan_capacity, const float* sink, int32_t dtype,
                             int32_t* status, void* stream);

/* b200_paged_decode_gqa with an attention sink (as above) and value heads of a size of their own.  Workspace:
 * b200_paged_decode_gqa_workspace_bytes() with head_dim_qk. */
int b200_paged_decode_sink(const void* q, const void* k_cache, const void* v_cache, void* out,
                           const int32_t* block_tables, int64_t bt_stride, const int64_t* context_lens, int32_t batch,
                           int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk, int32_t head_dim_v,
                           int32_t block_size, int64_t num_blocks, float scale, const float* sink, void* workspace,
                           size_t workspace_bytes, int32_t dtype, int32_t* status, void* stream);

/* One sublayer boundary of a decoder that norms the sublayer's output, fp32 residual x [rows, d] in place:
 *   x <- x + y / sqrt(mean(y^2) + eps) * norm_w,  h = x, or h = x / sqrt(mean(x^2) + eps) * final_w if given.
 * With embed [vocab, d] / tokens [rows] the residual starts as the embedding row instead.  y, h, embed in dtype. */
int b200_residual_norm(float* x, const int64_t* tokens, const void* embed, int64_t vocab, const void* y,
                       const float* norm_w, const float* final_w, float eps, void* h, int64_t rows, int32_t d,
                       int32_t dtype, int32_t* status, void* stream);

/* Attention prologue with a norm per head: q [T, Hq, dim_k], k [T, Hkv, dim_k], v [T, Hkv, dim_v] are views of one
 * projection (token stride, heads contiguous).  q and k heads are divided by their root mean square (eps inside) and
 * multiplied by the fp32 weights [dim_k]; the channel pairs (2i, 2i + 1), i < rot_dims / 2, then turn by
 * positions[t] * freq[i] (freq fp64, device).  Writes q_out [T, Hq, dim_k], k_out [T, Hkv, dim_k] and, if caches are given,
 * k and v rows at slot_mapping (< 0: skipped).  dim_k <= 512. */
int b200_head_norm_rope_store(const void* q, const void* k, const void* v, int64_t token_stride, const float* q_norm_w,
                              const float* k_norm_w, float eps, const double* freq, int32_t rot_dims,
                              const int64_t* positions, void* q_out, void* k_out, void* k_cache, void* v_cache,
                              const int64_t* slot_mapping, int64_t num_slots, int64_t num_tokens, int32_t num_q_heads,
                              int32_t num_kv_heads, int32_t dim_k, int32_t dim_v, int32_t dtype, int32_t* status,
                              void* stream);

/* Latent rows without a rotary part: rows_out[t] = rows_in[t] / sqrt(mean + eps) * norm_w [rank], also written to
 * cache[slot_mapping[t]] (cache NULL: not stored). */
int b200_latent_norm_store(const void* rows_in, int64_t in_stride, const float* norm_w, float eps, void* rows_out,
                           void* cache, const int64_t* slot_mapping, int64_t num_slots, int64_t num_tokens, int32_t rank,
                           int32_t dtype, int32_t* status, void* stream);

/* Packs the cached rows of whole contexts: out row cu_seqlens_k[s] - cu_seqlens_k[0] + j = pool row of position j of
 * sequence s.  cache [num_blocks, block_size] rows of row_bytes bytes. */
int b200_gather_rows(const void* cache, int32_t block_size, int64_t num_blocks, int64_t row_bytes,
                     const int32_t* block_tables, int64_t bt_stride, const int32_t* cu_seqlens_k, int32_t num_seqs,
                     int32_t max_seqlen_k, void* out, int64_t out_rows, int32_t* status, void* stream);

/* o <- o * sigmoid(gate), element by element, in place; o contiguous [rows, width], gate with a row stride. */
int b200_sigmoid_gate(void* o, const void* gate, int64_t gate_stride, int64_t rows, int32_t width, int32_t dtype,
                      void* stream);
/* x <- max(x, 0)^2 in place. */
int b200_squared_relu(void* x, int64_t n, int32_t dtype, void* stream);
/* z <- cap tanh(scale z / cap) in place (cap <= 0: scale z). */
int b200_softcap_logits(float* logits, int64_t n, float scale, float cap, void* stream);

/* Gated delta rule over per-sequence fp32 states [num_slots, num_heads, dim_k, dim_v]; value head h uses key head
 * h / (num_heads / num_k_heads).  With q^, k^ of unit length (1e-6 inside the root; q^ also times dim_k^-1/2),
 * beta = sigmoid(b), g = exp(-exp(a_log) softplus(a_in + dt_bias)):
 *   S <- g S,  u = beta (v - S^T k^),  S <- S + k^ u^T,  o = S^T q^,
 *   out = o / sqrt(mean(o^2) + eps) * norm_w [dim_v] * silu(gate)
 * q, k, v are projections behind a causal convolution per channel over `taps` tokens and silu.
 *
 * b200_delta_conv: that convolution for ragged portions; x [tokens, width] (token stride) -> out [tokens, width]; weights
 * fp32 [taps, width], the last row weighs the current token.  ring fp32 [num_slots, taps, width] keeps the input of
 * position p in row p mod taps and is moved on.  width a multiple of 4, pointers 16-byte aligned.
 * b200_delta_rule: ragged portions behind b200_delta_conv (q, k, v with act_stride; b, a_in [T, num_heads] and gate
 * [T, num_heads * dim_v] with proj_stride).  bf16 with dim_k, dim_v multiples of 16 up to 128 runs the chunked
 * tensor-core kernels (workspace: b200_delta_rule_workspace_bytes(); without one, tokens go in order).
 * b200_delta_step: one token per sequence, context_lens[i] long with it (0: skipped), straight from the projections
 * (one row stride), convolution included; col_q / col_k / col_v: columns of q / k / v in conv_w and the ring.
 * Slots < 0 are skipped; a sequence whose first token of the call is at position 0 starts from zero. */
int b200_delta_conv(const void* x, int64_t token_stride, const float* weights, int32_t taps, int32_t width, float* ring,
                    int64_t num_slots, const int64_t* state_slots, const int32_t* cu_seqlens_q,
                    const int32_t* cu_seqlens_k, int32_t num_seqs, int64_t total_tokens, void* out, int32_t dtype,
                    int32_t* status, void* stream);
size_t b200_delta_rule_workspace_bytes(int32_t num_seqs, int64_t total_tokens, int32_t num_heads, int32_t dim_k,
                                       int32_t dim_v, int32_t dtype);
int b200_delta_rule(const void* q, const void* k, const void* v, int64_t act_stride, const void* b, const void* a_in,
                    const void* gate, int64_t proj_stride, const float* dt_bias, const float* a_log, const float* norm_w,
                    float eps, float* state, int64_t num_slots, const int64_t* state_slots, const int32_t* cu_seqlens_q,
                    const int32_t* cu_seqlens_k, int32_t num_seqs, int64_t total_tokens, int32_t num_heads,
                    int32_t num_k_heads, int32_t dim_k, int32_t dim_v, void* out, void* workspace, size_t workspace_bytes,
                    int32_t dtype, int32_t* status, void* stream);
int b200_delta_step(const void* q, const void* k, const void* v, const void* b, const void* a_in, const void* gate,
                    int64_t proj_stride, const float* conv_w, int32_t taps, int32_t conv_width, int32_t col_q,
                    int32_t col_k, int32_t col_v, float* conv_ring, const float* dt_bias, const float* a_log,
                    const float* norm_w, float eps, float* state, int64_t num_slots, const int64_t* state_slots,
                    const int64_t* context_lens, int32_t num_seqs, int32_t num_heads, int32_t num_k_heads, int32_t dim_k,
                    int32_t dim_v, void* out, int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Mechanisms of decoders with parallel gated sublayers, windowed latent attention with sinks, grouped expert routing and
 * per-layer token inputs (the Meresun family; the reference has no counterpart).  All constants are parameters.
 * ------------------------------------------------------------------------------------------- */

/* b200_residual_norm with an embedding row that may also join an existing residual, and a norm in equal parts of the row:
 *   x <- (start ? 0 : x) + y / sqrt(mean(y^2) + eps) * y_norm_w + embed_scale embed[tokens]     (y, embed: NULL = absent)
 *   h  = x / sqrt(mean over the channel's part of x^2 + eps) * norm_w, `groups` consecutive parts; norm_w NULL: h = x. */
int b200_residual_group_norm(float* x, const void* y, const float* y_norm_w, const int64_t* tokens, const void* embed,
                             int64_t vocab, float embed_scale, int32_t start, const float* norm_w, int32_t groups, float eps,
                             void* h, int64_t rows, int32_t d, int32_t dtype, int32_t* status, void* stream);

/* Parallel sublayers into the fp32 residual x [rows, d], in place: x <- x + y1 sigmoid(gate1) + y2 sigmoid(gate2), h = x in
 * dtype.  y1, y2 contiguous [rows, d] in dtype, gates with one row stride; y2 NULL: one sublayer.  top_k > 0: y2 holds expert
 * rows [rows * top_k, d] and row t takes sum_k row_weight[t, k] y2[slot_to_row[t, k]]. */
int b200_gated_residual(float* x, const void* y1, const void* gate1, const void* y2, const void* gate2, int64_t gate_stride,
                        const float* row_weight, const int32_t* slot_to_row, int32_t top_k, void* h, int64_t rows, int32_t d,
                        int32_t dtype, int32_t* status, void* stream);

/* out = c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 per row of z [rows, width] (row stride), coef fp32 [4] on the device,
 * N(u) = u / sqrt(mean(u^2) + eps), powers element by element; out contiguous. */
int b200_poly_norm(const void* z, int64_t row_stride, const float* coef, float eps, void* out, int64_t rows, int32_t width,
                   int32_t dtype, void* stream);

/* out[t] = gelu_tanh(u[t]) * table[tokens[t], first .. first + width - 1]; u, out [rows, width], table [vocab, table_width]. */
int b200_gelu_table(const void* u, const void* table, int64_t table_width, int64_t vocab, int32_t first, const int64_t* tokens,
                    void* out, int64_t rows, int32_t width, int32_t dtype, int32_t* status, void* stream);

/* Latent attention with a rotary part, between the down-projections and the rest, one launch:
 *   q_out[t]  = q_in[t] / rms * q_norm_w [q_rank]                                            (q_in NULL: no query latent)
 *   kv_out[t] = [kv_in[t, :kv_rank] / rms * kv_norm_w | rotated kv_in[t, kv_rank:]], also written to cache[slot_mapping[t]]
 * The channel pairs (2i, 2i + 1), i < rot_dims / 2, of the rotary part (rope_dim wide) turn by positions[t] * freq[i] (freq
 * fp64); cos and sin are multiplied by `magnitude`.  Inputs with row strides, outputs contiguous. */
int b200_latent_prologue(const void* q_in, int64_t q_stride, const float* q_norm_w, int32_t q_rank, void* q_out,
                         const void* kv_in, int64_t kv_stride, const float* kv_norm_w, int32_t kv_rank, int32_t rope_dim,
                         float eps, const double* freq, int32_t rot_dims, float magnitude, const int64_t* positions,
                         void* kv_out, void* cache, const int64_t* slot_mapping, int64_t num_slots, int64_t num_tokens,
                         int32_t dtype, int32_t* status, void* stream);

/* The same rotation on the last rope_dim channels of every head of q [num_tokens, num_heads, head_dim], in place; the rotated
 * parts of the first tail_rows tokens are also written to tail [tail_rows, num_heads, rope_dim]. */
int b200_rotate_heads(void* q, int64_t num_tokens, int32_t num_heads, int32_t head_dim, int32_t rope_dim, const double* freq,
                      int32_t rot_dims, float magnitude, const int64_t* positions, void* tail, int64_t tail_rows, int32_t dtype,
                      void* stream);

/* b200_gather_rows for the ends of contexts: sequence s is cu_seqlens_full[s + 1] - cu_seqlens_full[s] tokens long and its last
 * cu_seqlens_k[s + 1] - cu_seqlens_k[s] rows are packed (cu_seqlens_full NULL: whole contexts).  Rows of out (out_rows of them)
 * behind the last packed one become zero. */
int b200_gather_last_rows(const void* cache, int32_t block_size, int64_t num_blocks, int64_t row_bytes,
                          const int32_t* block_tables, int64_t bt_stride, const int32_t* cu_seqlens_k,
                          const int32_t* cu_seqlens_full, int32_t num_seqs, int32_t max_seqlen_k, void* out, int64_t out_rows,
                          int32_t* status, void* stream);

/* Packed ragged causal attention with keys in two parts, a sliding window and a sink: query i of a sequence (at the end of its
 * k_len keys, bottom-right aligned) sees keys j with 0 <= (k_len - q_len + i) - j < window (window 0: all earlier ones).
 * k_head [total_k, num_kv_heads, head_dim_qk - tail_dim] and k_tail [total_k, tail_dim], the last columns of every head's key
 * (tail_dim 0: none); sink as in b200_prefill_varlen_sink.  plan: tile list for b200_prefill_window_tile_rows() rows, or NULL.
 * bf16: tcgen05 kernels for 192/128 (tail 64 or 0) and 128/128, mma.sync for multiples of eight up to 192/128; else general. */
int32_t b200_prefill_window_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk, int32_t tail_dim,
                                      int32_t head_dim_v, int32_t dtype);
int b200_prefill_varlen_window(const void* q, const void* k_head, const void* k_tail, const void* v, void* out,
                               int64_t q_token_stride, int64_t k_head_token_stride, int64_t k_tail_token_stride,
                               int64_t v_token_stride, int64_t total_q_tokens, int64_t total_k_tokens,
                               const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, int32_t num_seqs,
                               int32_t max_seqlen_q, int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk,
                               int32_t tail_dim, int32_t head_dim_v, float scale, int32_t window, const float* sink,
                               const int32_t* plan, int32_t plan_tile_rows, int32_t plan_capacity, int32_t dtype,
                               int32_t* status, void* stream);

/* b200_mla_decode over the last `window` tokens of every context (0: all) with exp(sink[h]) in the softmax denominator (sink
 * fp32 [num_heads] or NULL).  Workspace as b200_mla_decode. */
int b200_mla_decode_window(const void* q_abs, const void* q_rope, const void* latent_cache, void* out_latent,
                           const int32_t* block_tables, int64_t bt_stride, const int64_t* context_lens, int32_t batch,
                           int32_t num_heads, int32_t kv_lora_rank, int32_t rope_dim, int32_t block_size, int64_t num_blocks,
                           float scale, int32_t window, const float* sink, void* workspace, size_t workspace_bytes,
                           int32_t dtype, int32_t* status, void* stream);

/* Routing with a choice correction and groups: s = sigmoid(logits), c = s + correction (all fp32).  Experts form `groups` equal
 * groups of neighbours; a group's score is the sum of its two largest c, the `keep` best groups stay, and of their experts the
 * `top` with the largest c are chosen.  weight [tokens, top] = s of the chosen / (their sum + 1e-20).  sorted_token [tokens *
 * top] lists the tokens of the rows grouped by expert, expert_offsets [experts] their exclusive ends, slot_to_row [tokens, top]
 * the row of a token's k-th choice.  At most 512 experts, top 32, 64 groups. */
size_t b200_moe_group_route_workspace_bytes(int32_t num_tokens, int32_t num_experts, int32_t top);
int b200_moe_group_route(const float* logits, const float* correction, int32_t num_tokens, int32_t num_experts, int32_t top,
                         int32_t groups, int32_t keep, int32_t* sorted_token, float* weight, int32_t* expert_offsets,
                         int32_t* slot_to_row, void* workspace, size_t workspace_bytes, void* stream);

/* b200_moe_grouped_gemm without biases, for any size and also fp32 (general kernel).  act: what follows the linear map —
 * nothing; the clamped GLU: w [experts, 2 n_out, k_dim] = [gate | up] and out = g sigmoid(slope g) (u + 1) with g =
 * min(gate, limit), u = clamp(up, -limit, limit); the squared ReLU max(., 0)^2 (of the fp32 sums).  limit and slope count for
 * the GLU only.
 * flags: 0 or B200_MOE_GEMM_EARLY_LAUNCH. */
#define B200_EXPERT_LINEAR 0
#define B200_EXPERT_CLAMPED_GLU 1
#define B200_EXPERT_SQUARED_RELU 2
int b200_moe_grouped_linear(const void* x, const void* w, void* out, const int32_t* expert_offsets, int64_t num_rows,
                            int32_t num_experts, int32_t n_out, int32_t k_dim, int32_t act, float limit, float slope,
                            int32_t flags, int32_t dtype, int32_t* status, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Mechanisms of decoders with token shift, short convolutions in front of attention, sigmoid attention inside chunks and a
 * softmax over the chosen experts (the Sodonex family; the reference has no counterpart).  All constants are parameters.
 *
 * State slots: with cu_seqlens_q / cu_seqlens_k (int32 [num_seqs + 1]) a step holds ragged portions, the last tokens of contexts
 * of cu_seqlens_k lengths, and rows behind the last sequence are padding; with cu_seqlens_q NULL row i is sequence i with
 * context_lens[i] tokens (0: padding).  state_slots int64 [num_seqs], -1: no state.  A sequence at position 0 ignores what its
 * slot holds; every call moves the state on.
 * ------------------------------------------------------------------------------------------- */

/* One boundary between sublayers: x' = x + gain y / sqrt(mean(y^2) + eps), or embed_scale embed[tokens] where embed is given
 * (y NULL: x' = x).  top > 0: y holds expert rows [rows * top, d] and row t takes sum_k row_weight[t, k] y[slot_to_row[t, k]].
 * x' goes to x_out (NULL: nowhere; x_out == x is allowed without shift), and h [rows, d] in dtype is one of
 *   x' + (before - x') shift    shift fp32 [d]; before = the previous token's x', from state [num_slots, d] at a portion's start
 *   final_gain x' / sqrt(mean(x'^2) + eps)    final_norm
 *   x'                                        otherwise */
int b200_shift_residual(const float* x, float* x_out, const int64_t* tokens, const void* embed, int64_t vocab, float embed_scale,
                        const void* y, const float* row_weight, const int32_t* slot_to_row, int32_t top, float gain,
                        const float* shift, float* state, int64_t num_slots, const int64_t* state_slots,
                        const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const int64_t* context_lens, int32_t num_seqs,
                        int32_t final_norm, float final_gain, float eps, void* h, int64_t rows, int32_t d, int32_t dtype,
                        int32_t* status, void* stream);

/* Attention prologue: causal convolution of `taps` taps on every channel of q [T, Hq * D] and k [T, Hkv * D] (one token stride;
 * weights [taps, channels], the last row weighs the current token), v = the convolved k, RMS norm of the whole convolved q and of
 * the whole convolved k, rotation of the first rot_dims channels of every head (channel i with i + rot_dims / 2, by positions[t] *
 * freq[i], freq fp64).  q_out [T, Hq, D]; k_out, v_out [T, Hkv, D] (NULL: not wanted); k and v also go to the pools at
 * slot_mapping[t] (negative: not stored).  ring [num_slots, taps - 1, (Hq + Hkv) * D] keeps the last inputs of every sequence. */
int b200_conv_norm_rope_store(const void* q, const void* k, int64_t token_stride, const float* conv_q, const float* conv_k,
                              int32_t taps, float* ring, int64_t num_slots, const int64_t* state_slots,
                              const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const int64_t* context_lens,
                              int32_t num_seqs, const float* q_norm_w, const float* k_norm_w, float eps, const double* freq,
                              int32_t rot_dims, const int64_t* positions, void* q_out, void* k_out, void* v_out, void* k_cache,
                              void* v_cache, const int64_t* slot_mapping, int64_t pool_slots, int64_t num_tokens,
                              int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim, int32_t dtype, int32_t* status,
                              void* stream);

/* Packed ragged causal attention with weights sigmoid(scale q.k + bias[head]) that are summed as they are.  Query i of a sequence
 * (at the end of its k_len keys) has index n = k_len - q_len + i and sees the keys j <= n with j / chunk = n / chunk (chunk 0:
 * all): packed contexts start at a multiple of the chunk.  out[t, h] is multiplied by sigmoid(gate[t, h]) (gate NULL: not).
 * plan: tile list for b200_sigmoid_attention_tile_rows() rows, or NULL.  bf16: tcgen05 kernel for 128/128 and 64/64, mma.sync for
 * multiples of eight up to 192/128; else general. */
int32_t b200_sigmoid_attention_tile_rows(int32_t num_q_heads, int32_t num_kv_heads, int32_t head_dim_qk, int32_t head_dim_v,
                                         int32_t dtype);
int b200_sigmoid_attention(const void* q, const void* k, const void* v, void* out, int64_t q_token_stride, int64_t k_token_stride,
                           int64_t v_token_stride, int64_t total_q_tokens, int64_t total_k_tokens, const int32_t* cu_seqlens_q,
                           const int32_t* cu_seqlens_k, int32_t num_seqs, int32_t max_seqlen_q, int32_t num_q_heads,
                           int32_t num_kv_heads, int32_t head_dim_qk, int32_t head_dim_v, float scale, const float* bias,
                           int32_t chunk, const void* gate, int64_t gate_token_stride, const int32_t* plan,
                           int32_t plan_tile_rows, int32_t plan_capacity, int32_t dtype, int32_t* status, void* stream);

/* The same for one token per sequence over the paged pools: the last token of context_lens[i] sees its own chunk.  Workspace as
 * b200_paged_decode_gqa. */
int b200_sigmoid_decode(const void* q, const void* k_cache, const void* v_cache, void* out, const int32_t* block_tables,
                        int64_t bt_stride, const int64_t* context_lens, int32_t batch, int32_t num_q_heads, int32_t num_kv_heads,
                        int32_t head_dim_qk, int32_t head_dim_v, int32_t block_size, int64_t num_blocks, float scale,
                        const float* bias, int32_t chunk, const void* gate, int64_t gate_token_stride, void* workspace,
                        size_t workspace_bytes, int32_t dtype, int32_t* status, void* stream);

/* b200_moe_group_route without groups, on z = logits + bias: the `top` largest z are chosen (equal ones: the lower index), their
 * weights are the softmax of z over the chosen.  Workspace as b200_moe_group_route. */
int b200_moe_softmax_route(const float* logits, const float* bias, int32_t num_tokens, int32_t num_experts, int32_t top,
                           int32_t* sorted_token, float* weight, int32_t* expert_offsets, int32_t* slot_to_row, void* workspace,
                           size_t workspace_bytes, void* stream);

/* ---------------------------------------------------------------------------------------------
 * Diagnostic (no counterpart in the reference, which has no device code): runs the give-up path of the
 * bounded barrier waits that the tcgen05 / TMA kernels share.  One CTA holds tensor memory, arms a barrier
 * that can never complete, and waits on it from two threads: one with `poll_limit` polls (1..65536), one
 * with the kernels' default limit.  Nothing faults and nothing loops without bound.  Afterwards
 *   result[0] = 0 and result[1] = poll_limit : the short wait ran out at its limit,
 *   result[2] = 0 and result[3] < 2^22       : the other wait left through the CTA's abort flag,
 *   result[4] = 1                            : tensor memory was allocated and has been freed,
 * and *status holds B200_ERR_TIMEOUT (read and clear it with b200_read_status).  result: device int32[5].
 * ------------------------------------------------------------------------------------------- */
int b200_selftest_bounded_wait(int32_t poll_limit, int32_t* result, int32_t* status, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* B200LLM_H_ */
