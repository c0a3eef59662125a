/*
 * minivllm_b200 — C ABI of the B200 (sm_100a) ragged-batch attention path.
 *
 * Every entry point is `extern "C"`, takes plain device pointers, sizes and a
 * CUDA stream handle (a `cudaStream_t` passed as `void*`), launches on that
 * stream without synchronising the host, and returns an `int` status:
 * 0 = launched, non-zero = rejected before any launch (see mv_status).
 * The library allocates no device memory on these paths and keeps no pointer
 * after a call returns; the caller owns inputs, outputs and scratch.
 *
 * Each declaration cites the function of the reference engine
 * (Wenyueh/MinivLLM, paths relative to that project) whose work it does.
 */
#ifndef MINIVLLM_B200_H
#define MINIVLLM_B200_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

/* Element types of activations, weights and of a non-quantised cache (each entry point says which it takes). */
enum mv_dtype { MV_F16 = 0, MV_BF16 = 1, MV_F32 = 2 };

/* What a gate g does to the value u beside it.  GELU_TANH: the tanh form of gelu.  CLAMPED (with a limit):
 * g' sigmoid(1.702 g') (u' + 1) with g' = min(g, limit), u' = u clamped to +-limit. */
enum mv_act { MV_ACT_NONE = -1, MV_ACT_SIGMOID = 0, MV_ACT_SILU = 1, MV_ACT_GELU_TANH = 2, MV_ACT_CLAMPED = 3, MV_ACT_RELU = 4 };

enum mv_status {
  MV_OK = 0,
  MV_ERR_NULL = 1,        /* a required pointer is null */
  MV_ERR_ALIGN = 2,       /* a pointer or stride breaks the 16-byte rule */
  MV_ERR_SHAPE = 3,       /* unsupported head_dim / head ratio / negative size */
  MV_ERR_WORKSPACE = 4,   /* scratch buffer too small */
  MV_ERR_DTYPE = 5,
  MV_ERR_CUDA = 6,        /* the launch itself reported an error */
  MV_ERR_LIMIT = 7        /* size beyond a documented fixed maximum */
};

/* Text of the last non-zero status returned on the calling thread. */
const char* mv_last_error_string(void);

/* Library version, bumped when a signature changes. */
int mv_abi_version(void);

/*
 * Scatter new K/V rows into the paged cache.
 * Replaces: src/myvllm/layers/attention.py:67-108 `store_kvcache` and its
 * Triton kernel :7-64.  For every token t with slot_mapping[t] >= 0:
 *   k_cache[slot_mapping[t]] = key[t],  v_cache[slot_mapping[t]] = value[t]
 * with the cache seen as (num_slots, num_kv_heads, head_dim); slot -1 (any
 * negative) is skipped.  key/value are (num_tokens, num_kv_heads, head_dim)
 * with an arbitrary token stride (in elements) so the split view of a fused
 * qkv projection needs no copy; heads and head_dim are contiguous.
 *
 * When k_scale and v_scale are non-null the caches hold int8 codes and the
 * scatter is fused with per-token-per-head symmetric quantisation (no
 * counterpart in the reference, which has no quantisation):
 *   amax = max|x| over head_dim (fp32); s = float(fp16(amax / 127));
 *   code = clamp(rint(x / s), -127, 127), 0 when s == 0;
 * codes go to (num_slots, num_kv_heads, head_dim) int8 and s, as fp16, to
 * (num_slots, num_kv_heads).
 */
int mv_store_kvcache(const void* key, const void* value,
                     int64_t k_stride_tok, int64_t v_stride_tok,
                     void* k_cache, void* v_cache,
                     void* k_scale, void* v_scale,
                     const int64_t* slot_mapping,
                     int64_t num_tokens, int64_t num_slots,
                     int num_kv_heads, int head_dim,
                     int dtype, void* stream);

/*
 * Bytes of scratch mv_paged_decode needs for the given problem (split-K
 * partial results); depends on shapes only, never on context_lens values.
 * Returns -1 for an invalid shape.
 * The first 64 KiB of the scratch hold arrival counters (which piece of a
 * split sequence was written last): they must be ZERO when the buffer is
 * first used, and every call leaves them zero, so fill the buffer with zeros
 * once when it is allocated.  One buffer may serve calls of any shapes, one
 * at a time (calls that overlap on the GPU need buffers of their own).
 */
int64_t mv_paged_decode_workspace_bytes(int batch, int num_heads,
                                        int num_kv_heads, int head_dim,
                                        int max_blocks, int block_size);

/*
 * One-query-per-sequence attention over the paged cache.
 * Replaces: src/myvllm/layers/attention.py:418-473 `paged_attention_decode`
 * and its Triton kernel :283-415.  For sequence b and query head h:
 *   out[b,h] = softmax_j(scale * q[b,h] . K[b,j,h/G]) . V[b,j,h/G],  j < context_lens[b]
 * where token j lives at cache[block_tables[b, j / block_size], j % block_size]
 * and G = num_heads / num_kv_heads.  Tokens whose table entry is negative
 * get zero weight; a row with no live token writes zeros.
 * q/out are (batch, num_heads, head_dim) contiguous; caches are
 * (num_blocks, block_size, num_kv_heads, head_dim) contiguous, of `dtype`,
 * or int8 codes with fp16 scales (num_blocks, block_size, num_kv_heads)
 * when k_scale/v_scale are non-null.  block_tables is (batch, max_blocks)
 * int32 with row stride bt_stride; context_lens is int32 or int64 and is
 * clamped to [0, max_blocks * block_size].
 * The grid depends on shapes only, so the call can be captured in a graph.
 * batch * max_blocks * block_size must stay below 2^31 (status 7 otherwise).
 * The KV tokens of the whole batch are divided evenly among the thread
 * blocks, so where a long sequence is cut depends on the other sequences:
 * a row's result can differ in its last bits between batch compositions.
 */
int mv_paged_decode(void* out, const void* q,
                    const void* k_cache, const void* v_cache,
                    const void* k_scale, const void* v_scale,
                    const int32_t* block_tables, int64_t bt_stride,
                    int max_blocks,
                    const void* context_lens, int ctx_is_i64,
                    int batch, int num_heads, int num_kv_heads, int head_dim,
                    int block_size, int64_t num_blocks, float scale,
                    void* workspace, int64_t workspace_bytes,
                    int dtype, void* stream);

/*
 * mv_paged_decode for callers that cannot allocate device memory.
 * No counterpart in the reference (its Triton decode kernel needs no scratch
 * because it never splits a sequence).  Same arguments and results as
 * mv_paged_decode without `workspace`: the split-K scratch is a fixed array of
 * mv_paged_decode_static_capacity() bytes (8 MiB) inside the library's device
 * image, held by every GPU that loads the library.  Meant for a serving
 * process that gave all free HBM to the KV pool and forbids later
 * allocation, for latency-critical loops where the allocator must not run,
 * and for bindings that only pass inputs and outputs (not for CUDA host
 * callbacks: no launch may be made from one).
 * A problem needing more scratch than the array holds returns MV_ERR_LIMIT
 * and launches nothing.  All calls on a device share the array: calls that
 * overlap on the GPU race, so keep them on one stream or order them.  The
 * first call on each device resolves the array's address (a host-side lookup)
 * and should be made before any stream capture, from one host thread; the
 * address is stale after a cudaDeviceReset.  Neither function calls
 * cudaMalloc, cudaFree or any allocating library routine.
 */
int64_t mv_paged_decode_static_capacity(void);
int mv_paged_decode_static(void* out, const void* q,
                           const void* k_cache, const void* v_cache,
                           const void* k_scale, const void* v_scale,
                           const int32_t* block_tables, int64_t bt_stride,
                           int max_blocks,
                           const void* context_lens, int ctx_is_i64,
                           int batch, int num_heads, int num_kv_heads,
                           int head_dim, int block_size, int64_t num_blocks,
                           float scale, int dtype, void* stream);

/*
 * Varlen causal prefill attention over a packed ragged batch.
 * Replaces: src/myvllm/layers/attention.py:212-280 `flash_attention_prefill`
 * and its Triton kernel :111-209.  Sequence s owns rows
 * [cu_seqlens[s], cu_seqlens[s+1]) of q/k/v; row i attends to rows <= i of
 * its own sequence; query head h reads kv head h / (num_heads/num_kv_heads).
 * q/out are (total_tokens, num_heads, 128), k/v (total_tokens, num_kv_heads,
 * 128); q/k/v take a token stride in elements (heads dense within a token),
 * out is contiguous.  fp32 accumulation on the tcgen05 tensor cores.
 * No host synchronisation: the grid is an upper bound computed from
 * total_tokens and num_seqs, or (up to 320 sequences) one block per SM that
 * takes query tiles from a work counter inside the library; a launch uses
 * the next of 1,024 counters and leaves it zeroed, nothing is allocated.
 * error_word points to one zero-initialised int in device memory that the
 * caller keeps: a kernel wait that runs out of time stores a non-zero code
 * there (and later launches return at once until the caller clears it).
 */
int mv_prefill_varlen(void* out, const void* q, const void* k, const void* v,
                      int64_t q_stride_tok, int64_t k_stride_tok,
                      int64_t v_stride_tok, const int32_t* cu_seqlens,
                      int num_seqs, int64_t total_tokens, int num_heads,
                      int num_kv_heads, int head_dim, float scale,
                      int* error_word, int dtype, void* stream);

/*
 * Prefill attention with a cached prefix (or a chunk of a longer prompt):
 * the queries are the packed UNCACHED tokens (cu_seqlens_q), the keys and
 * values are read from the paged cache through block_tables, which must
 * already hold every token of the step (store_kvcache first).  Sequence s has
 * k_s = cu_seqlens_k[s+1]-cu_seqlens_k[s] keys and q_s queries; query i sits
 * at position k_s - q_s + i and attends to keys at positions <= its own.
 * This is the case the reference prepares (src/myvllm/engine/model_runner.py
 * :198-215 builds cu_seqlens_k != cu_seqlens_q and block_tables on a prefix
 * hit) but never computes: its prefill kernel indexes K/V with the query
 * offsets (src/myvllm/layers/attention.py:135-137,171,194).  block_size must
 * divide 128 (multiple of 8) or be a multiple of 128.  Same error_word
 * contract as mv_prefill_varlen.
 * Precondition: every row of every cache block that a table names must hold
 * FINITE values, also the rows past a sequence's last key (the rest of its
 * last block) and block 0 (read in place of a missing table entry).  Such
 * rows get weight exactly 0, but their V values still pass through the
 * tensor-core product, and 0 x NaN or 0 x Inf is NaN.  Allocate the pool
 * zero-initialised (the engine does); blocks that were used before hold
 * finite stale values and are fine.  mv_paged_decode has no such
 * precondition (it zero-fills rows it does not use).
 */
int mv_prefill_paged(void* out, const void* q, int64_t q_stride_tok,
                     const void* k_cache, const void* v_cache,
                     const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                     const int32_t* block_tables, int64_t bt_stride,
                     int max_blocks, int block_size, int64_t num_blocks,
                     int num_seqs, int64_t total_q_tokens, int num_heads,
                     int num_kv_heads, int head_dim, float scale,
                     int* error_word, int dtype, void* stream);

/*
 * Per-step metadata, built on the GPU from persistent per-sequence state.
 * State (device memory, owned by the caller, one row per sequence "slot"):
 *   tables (num_slots, max_blocks) int32 block table rows, -1 = none;
 *   seq_len_state (num_slots) int32 tokens already in the cache;
 *   last_token_state (num_slots) int64 last sampled token.
 *
 * mv_build_decode_meta replaces src/myvllm/engine/model_runner.py:231-256
 * `prepare_decode` (and the per-layer positions of models/qwen3.py:210-212):
 * for row b < *n_active with slot s and p = seq_len_state[s] it writes
 * input_ids[b] = last_token_state[s], positions[b] = p, context_lens[b] = p+1,
 * slot_mapping[b] = table[s][p/bs]*bs + p%bs, tables_out[b] = table[s], and
 * bumps seq_len_state[s]; rows b >= *n_active (graph padding) get 0/0/0/-1
 * and a table of -1.  n_active is read on the device so a captured graph can
 * be replayed with any batch up to batch_padded.  A slot may appear once.
 *
 * mv_build_prefill_meta replaces model_runner.py:180-227 `prepare_prefill`
 * (and qwen3.py:199-206): sequence i (slot seq_slots[i]) feeds tokens at
 * positions num_cached[i] .. seq_lens[i]-1 (num_cached may be null = 0);
 * writes cu_seqlens_q/k (num_seqs+1, int32), positions and slot_mapping
 * (total_tokens, int64), last_token_index (num_seqs, int64) and sets
 * seq_len_state[slot] = seq_lens[i].  total_tokens = sum of fed tokens.
 *
 * mv_update_block_tables applies `num_updates` (slot, index, block) int32
 * triples to the table state (a sequence gained a block, or was allocated).
 */
int mv_build_decode_meta(const int32_t* seq_slots, const int32_t* n_active,
                         int batch_padded, const int32_t* tables,
                         int64_t tables_stride, int max_blocks, int block_size,
                         int32_t* seq_len_state, const int64_t* last_token_state,
                         int64_t* input_ids, int64_t* positions,
                         int64_t* slot_mapping, int64_t* context_lens,
                         int32_t* tables_out, int64_t out_stride, void* stream);
int mv_build_prefill_meta(const int32_t* seq_slots, const int32_t* seq_lens,
                          const int32_t* num_cached, int num_seqs,
                          int64_t total_tokens, const int32_t* tables,
                          int64_t tables_stride, int max_blocks, int block_size,
                          int32_t* seq_len_state, int32_t* cu_seqlens_q,
                          int32_t* cu_seqlens_k, int64_t* positions,
                          int64_t* slot_mapping, int64_t* last_token_index,
                          void* stream);
int mv_update_block_tables(const int32_t* updates, int num_updates,
                           int32_t* tables, int64_t tables_stride,
                           int max_blocks, int num_slots, void* stream);

/*
 * Fused pre-attention step on the fused qkv projection output
 * qkv (tokens, (num_heads + 2*num_kv_heads) * 128), token stride in elements:
 * RMSNorm of every q and k head row (x * rsqrt(mean(x^2) + eps) * gamma,
 * rounded to the model dtype), rotate-half rotary embedding from fp32
 * cos/sin tables (max_position, 64) at positions[t], then q -> q_out
 * (tokens, num_heads, 128), k -> k_out (tokens, num_kv_heads, 128) and, when
 * slot_mapping is non-null, k and v -> the paged caches at slot_mapping[t]
 * (negative = skip), i.e. store_kvcache fused in.  With k_scale / v_scale
 * non-null the caches are int8 and the rows are quantised on the way in, with
 * the arithmetic and layouts of mv_store_kvcache (codes and fp16 scales equal
 * what mv_store_kvcache writes for k_out and v).
 * Replaces, in one launch: src/myvllm/models/qwen3.py:104-108 (rms_norm of q
 * and k, rotary_emb), layers/layernorm.py:10-17, layers/rotary_embedding.py
 * :4-23,77-83 and the store_kvcache call of layers/attention.py:498-510.
 */
int mv_qk_norm_rope_store(const void* qkv, int64_t qkv_stride_tok,
                          const int64_t* positions, const float* cos_table,
                          const float* sin_table, int max_position,
                          const void* gamma_q, const void* gamma_k, float eps,
                          void* q_out, void* k_out, void* k_cache,
                          void* v_cache, void* k_scale, void* v_scale,
                          const int64_t* slot_mapping,
                          int64_t num_slots, int64_t num_tokens, int num_heads,
                          int num_kv_heads, int head_dim, int dtype,
                          void* stream);

/*
 * Greedy sampling tail.  mv_argmax_rows reduces each row of a logits matrix
 * (rows, cols), row stride in elements, to one signed 64-bit key: high word =
 * the maximum logit in an integer form whose order is the float order (NaN
 * above +inf, as torch.argmax treats it), low word = 2^32-1 minus
 * (index_offset + column).  The larger key is the larger logit and, between
 * equal logits, the lower index, so vocabulary shards merge by an integer MAX
 * (e.g. an all-reduce of 8 bytes per row) -- mv_argmax_decode takes the
 * largest of `shards` keys per row, keys laid out (shards, rows), and writes
 * the token ids.  keys or tokens of mv_argmax_rows may be NULL; with tokens
 * set the decoded ids of this shard alone are written too (single-GPU path,
 * one launch).  Rows that start on 16-byte boundaries (aligned base, stride a
 * multiple of 8 elements) are read with 16-byte loads, others element-wise.
 * Replaces the gather of full-vocabulary logits to rank 0 and the argmax on
 * them: src/myvllm/layers/embedding_head.py:56-77 (ParallelLMHead.forward)
 * and src/myvllm/layers/sampler.py:15-19 in its greedy limit.
 */
int mv_argmax_rows(const void* logits, int64_t row_stride, int64_t rows,
                   int64_t cols, int64_t index_offset, int64_t* keys,
                   int64_t* tokens, int dtype, void* stream);
int mv_argmax_decode(const int64_t* keys, int shards, int64_t rows,
                     int64_t* tokens, void* stream);

/*
 * Temperature sampling tail, vocabulary-sharded.  Replaces the sampler
 * src/myvllm/layers/sampler.py:15-19 (logits / T, softmax, division by an
 * Exp(1) draw per entry, argmax) and the logits gather in front of it
 * (layers/embedding_head.py:56-77):  argmax_i p_i / E_i equals
 * argmax_i (logit_i / T - log E_i), which needs no softmax normaliser, so
 * every rank reduces its shard to the same 64-bit keys as mv_argmax_rows
 * (score in place of the logit) and the shards merge by integer MAX
 * (mv_argmax_decode).  E_i comes from Philox4x32-10 with key = seed and
 * counter = (global column / 4, row, *step): every rank and every
 * tensor-parallel degree draws the same noise for a given global column.
 * temperatures is (rows) fp32; a row with temperature 0 is greedy.  *step is
 * read on the device (a captured graph can advance it between replays).
 * mv_philox4x32_10 evaluates the generator on the host (for checking).
 */
int mv_sample_rows(const void* logits, int64_t row_stride, int64_t rows,
                   int64_t cols, int64_t index_offset,
                   const float* temperatures, uint64_t seed,
                   const int64_t* step, int64_t* keys, int64_t* tokens,
                   int dtype, void* stream);
int mv_philox4x32_10(uint64_t seed, uint64_t step, uint32_t row,
                     uint32_t column_group, uint32_t* out4);

/*
 * Tensor-parallel all-reduce over NVLink peer memory, fused with the residual
 * add and the RMSNorm that follow it.
 * Replaces: the `dist.all_reduce(result)` that ends every row-parallel linear
 * layer (src/myvllm/layers/linear.py:216-221, after o_proj and down_proj) plus
 * the residual add and RMSNorm each rank then repeats on the full activations
 * (src/myvllm/layers/layernorm.py:10-22, called from models/qwen3.py:187,215).
 *
 * A communicator owns, on every rank, one device allocation holding an INPUT
 * buffer (this rank's partial sums, written by the caller's GEMM), a GATHER
 * buffer (the normalised rows of all ranks, read by the caller's next GEMM)
 * and the barrier flags; peers map each other's allocation through CUDA IPC.
 * Set-up (once, allocates): every rank calls mv_comm_create, the caller
 * exchanges the mv_comm_handle_bytes()-byte handles of all ranks in rank order
 * (any host channel), every rank calls mv_comm_connect, and the caller makes
 * sure every rank has connected before the first launch (a host barrier).
 * `data_bytes` bounds rows*hidden*2 of one call; `timeout_ms` bounds every
 * in-kernel wait.
 *
 * mv_allreduce_residual_rmsnorm, with x_p (rows, hidden) in rank p's input
 * buffer and rank r owning rows [r*ceil(rows/N), min(rows, (r+1)*ceil(rows/N))):
 *   o = round(sum_p x_p[row]) (fp32, p ascending);
 *   residual_shard[row - first owned row] = round(residual_shard[...] + o);
 *   h[row] = round(residual * rsqrt(mean(residual^2) + eps) * gamma)
 * and h[row] is stored into the gather buffer of every rank.  The residual
 * stream stays sharded by rows: residual_shard is (owned rows, hidden) and may
 * be null on a rank that owns no row (rows < world).
 * Every rank must make the same sequence of calls with the same rows/hidden,
 * one call at a time per communicator (calls are ordered by the stream).
 * Launch-only (graph-capturable); peers are read and written with plain loads
 * and stores.  A wait that runs out of time stores a non-zero code in
 * *error_word (caller-owned device int, zero-initialised; 0x100|peer = partial
 * sums never arrived, 0x200|peer = result rows never arrived) and the kernel
 * returns; while the word is non-zero later launches return at once.  After
 * such an error the communicator must be reset on every rank (mv_comm_reset,
 * all ranks idle) before it is used again.
 *
 * mv_comm_create_emulated builds all N ranks on the current device; a call
 * then runs every rank in ONE cooperative launch (residual shard of rank p at
 * residual_shard + p*residual_slot_stride elements; mv_comm_input/output take
 * the rank as `slot`).  It exists to test the protocol on a single GPU (the
 * launch uses at most one block per SM in total).  On a real communicator
 * `slot` is 0 and residual_slot_stride is ignored.
 */
int64_t mv_comm_handle_bytes(void);
int mv_comm_create(int rank, int world, int64_t data_bytes, int timeout_ms,
                   void** comm_out, void* handle_out);
int mv_comm_connect(void* comm, const void* all_handles);
int mv_comm_create_emulated(int world, int64_t data_bytes, int timeout_ms,
                            void** comm_out);
int mv_comm_destroy(void* comm);
int mv_comm_reset(void* comm);
/* Caps the grid of the following mv_allreduce_residual_rmsnorm launches of this communicator (0 = no cap).  A
 * block of that kernel occupies a whole SM; a caller that keeps a second stream busy with GEMMs while a
 * bandwidth-bound call runs leaves them the remaining SMs this way.  Results do not depend on the grid. */
int mv_comm_set_max_blocks(void* comm, int max_blocks);
void* mv_comm_input(void* comm, int slot);
void* mv_comm_output(void* comm, int slot);
int mv_allreduce_residual_rmsnorm(void* comm, void* residual_shard,
                                  int64_t residual_slot_stride,
                                  const void* gamma, float eps, int rows,
                                  int hidden, int* error_word, int dtype,
                                  void* stream);
/* The same step (arguments, result, row ownership, error codes, bounded waits) with the two bulk transfers done
 * by the copy engines: barrier, cudaMemcpyAsync of the peers' partial rows of this rank's shard into staging
 * inside the communicator, one local kernel (the same sums and roundings), cudaMemcpyAsync of the normalised
 * rows to every peer, barrier.  For messages that are bound by the link (a prefill wave): the SMs stay free
 * while the bytes move, so another stream's work runs beside it.  Calls of both forms may follow each other on
 * one communicator. */
int mv_allreduce_residual_rmsnorm_staged(void* comm, void* residual_shard,
                                  int64_t residual_slot_stride,
                                  const void* gamma, float eps, int rows,
                                  int hidden, int* error_word, int dtype,
                                  void* stream);

/*
 * Single-rank form of the same step: for every row,
 *   s = x[row] (+ residual_in[row], rounded, when residual_in is non-null);
 *   out[row] = round(s * rsqrt(mean(s^2) + eps) * gamma);
 * and s is stored to residual_out[row - res_lo] for rows in [res_lo, res_hi)
 * (residual_out may be null; it may alias residual_in when res_lo is 0).
 * Replaces src/myvllm/layers/layernorm.py:10-28 (rms_forward and
 * residual_rms_forward).  x/out/residuals are (rows, hidden) contiguous.
 */
int mv_add_rmsnorm(void* out, const void* x, const void* residual_in,
                   void* residual_out, int64_t res_lo, int64_t res_hi,
                   const void* gamma, float eps, int64_t rows, int hidden,
                   int dtype, void* stream);

/*
 * SwiGLU activation on the fused gate_up projection output (rows, 2*inter),
 * row stride in elements: out[t, j] = silu(gu[t, j]) * gu[t, inter + j],
 * computed in fp32 and rounded once; out is (rows, inter) contiguous.
 * Replaces src/myvllm/layers/activation.py:17-20 (SiluAndMul.forward).
 */
int mv_silu_mul(void* out, const void* gate_up, int64_t gate_up_stride,
                int64_t rows, int inter, int dtype, void* stream);

/*
 * Steps between the sublayers of a decoder with an fp32 residual stream x (rows, width), updated in place, and RMS
 * norms over `groups` equal runs of channels.  dtype (MV_BF16 or MV_F32) is that of every void* operand; *_stride
 * are row strides in elements.  No counterpart in the reference.
 *   mv_embed_norm           x = embed[ids], or norm(embed[ids]) * w_post with w_post;  out = norm(x) * w_next, or x
 *                           without w_next (in all of these)
 *   mv_gated_residual_norm  y' = y * sigmoid(gate + gate_bias) (gate may be null);
 *                           x += mult * norm(y') * w_post;  out = norm(x) * w_next
 *   mv_moe_residual_norm    the same with y = sum_k top_weights[t, k] * expert_rows[pos[t, k]]
 *                           + sigmoid(shared_gate[t]) * shared[t]   (shared may be null)
 *   mv_pair_residual_norm   the same with y = (norm(a) * w_a + norm(b) * w_b) / 2, no gate
 *   mv_gated_group_norm     out = norm(y * silu(z)) * w
 *   mv_head_norm_gate       out = norm(y / den) * w * act(z) * mult, norms over `heads` equal runs; den (rows, heads) may be
 *                           null; w has one run's length, or the row's with full_weight; act MV_ACT_SILU or MV_ACT_SIGMOID;
 *                           out_stride 0: dense rows
 *   mv_gate_mul             out = gate applied to y (enum mv_act); a row of y is `heads` pieces y_head_stride
 *                           elements apart
 */
int mv_embed_norm(void* out, float* x, const int64_t* ids, const void* embed, int64_t vocab, const
    void* w_post, const void* w_next, int64_t rows, int width, int groups, float eps, int dtype, void* stream);
int mv_gated_residual_norm(void* out, float* x, const void* y, int64_t y_stride, const void* gate,
    int64_t gate_stride, const void* gate_bias, const void* w_post, const void* w_next, float mult,
    int64_t rows, int width, int groups, float eps, int dtype, void* stream);
int mv_moe_residual_norm(void* out, float* x, const void* expert_rows, const int32_t* pos, const
    float* top_weights, int top, const void* shared, int64_t shared_stride, const void* shared_gate,
    int64_t shared_gate_stride, const void* gate, int64_t gate_stride, const void* gate_bias, const
    void* w_post, const void* w_next, float mult, int64_t rows, int width, int groups, float eps,
    int dtype, void* stream);
int mv_pair_residual_norm(void* out, float* x, const void* a, int64_t a_stride, const void* w_a, const
    void* b, int64_t b_stride, const void* w_b, const void* w_post, const void* w_next, float mult,
    int64_t rows, int width, int groups, float eps, int dtype, void* stream);
int mv_head_norm_gate(void* out, int64_t out_stride, const void* y, int64_t y_stride, const float* den, const void* z,
    int64_t z_stride, const void* w, int full_weight, int act, float mult, int64_t rows, int width, int heads, float eps,
    int dtype, void* stream);
int mv_gated_group_norm(void* out, const void* y, int64_t y_stride, const void* z, int64_t z_stride,
    const void* w, int64_t rows, int width, int groups, float eps, int dtype, void* stream);
int mv_gate_mul(void* out, const void* y, int64_t y_stride, int64_t y_head_stride, int heads,
    const void* gate, int64_t gate_stride, int act, float limit, int64_t rows, int cols, int dtype, void*
    stream);

/*
 * Latent attention over a paged cache (num_blocks, block_size, rank + rot_dim) of rows [c | rotated key part].
 *   mv_latent_prep  down (tokens, rank + rot_dim, row stride): c = rms_norm(down[:rank]) * c_weight, rotary on the
 *                   shared key part and, in place, on the last rot_dim entries of every head of q (tokens,
 *                   heads * (dim + rot_dim)); rows go to latent_out (contiguous, may be null) and to cache[slot]
 *                   (slot < 0 skips).  cos/sin tables (max_position, rope_dims / 2) fp32.
 *   mv_latent_attention_rows  out[t, h] = sum_j softmax_j((q_lat . c_j + q_rot . k_j) * scale) c_j over keys
 *                   j <= positions[t] (token and head strides of out, q_lat and q_rot in elements), with exp(sink[h]) added to the denominator (sink may be null).  Token t belongs
 *                   to the sequence of cu_q (null: token t is row t of block_tables).  Any sizes up to rank 1,024.
 * dtype MV_BF16 or MV_F32.  No counterpart in the reference.
 */
int mv_latent_prep(void* q, int64_t q_stride, const void* down, int64_t down_stride, const void*
    c_weight, const int64_t* positions, const float* cos_table, const float* sin_table, int64_t
    max_position, void* latent_out, void* cache, const int64_t* slot_mapping, int64_t num_slots,
    int64_t tokens, int heads, int dim, int rot_dim, int rope_dims, int rank, float eps, int dtype,
    void* stream);
int mv_latent_attention_rows(void* out, int64_t out_stride, int64_t out_head_stride, const void* q_lat,
    int64_t q_lat_stride, int64_t q_lat_head_stride, const void* q_rot,
    int64_t q_rot_stride, int64_t q_rot_head_stride, const void* cache, const int32_t* block_tables,
    int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int32_t* cu_q, int
    num_seqs, const int64_t* positions, const void* sink, int64_t tokens, int heads, int rank, int
    rot_dim, float scale, int dtype, void* stream);

/*
 * State-space mixer over a packed batch.  Sequence s has tokens cu[s] .. cu[s + 1] (cu null: one token each), slot
 * slots[s] and start[s] earlier tokens; start 0 reads the slot as zeros, start < 0 marks a padding row.
 *   mv_conv_silu          out (tokens, channels) = silu(causal depthwise convolution of u with w (channels, taps))
 *   mv_conv_add           the same without silu, added to u
 *   mv_conv_state_update  state (num_slots, taps - 1, channels): the last inputs, oldest first
 *   mv_ssm_scan           xbc = [x: heads * vdim | B: groups * state_dim | C: the same] per token, dt before
 *                         bias and softplus; state (num_slots, heads, state_dim, vdim) fp32, updated
 * dtype MV_BF16 or MV_F32.  No counterpart in the reference.
 */
int mv_conv_silu(void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int
    taps, int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots, const
    int32_t* start, const void* state, int num_slots, int dtype, void* stream);
int mv_conv_add(void* out, const void* u, int64_t u_stride, const void* w, const void* bias, int
    taps, int channels, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t* slots, const
    int32_t* start, const void* state, int num_slots, int dtype, void* stream);
int mv_conv_state_update(void* state, const void* u, int64_t u_stride, int taps, int channels, const
    int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start, int num_slots, int dtype,
    void* stream);
int mv_ssm_scan(void* y, const void* xbc, const void* dt, int64_t dt_stride, const void* dt_bias,
    const void* A_log, const void* D, const int32_t* cu, int num_seqs, const int32_t* slots, const
    int32_t* start, float* state, int num_slots, int heads, int vdim, int state_dim, int groups, int
    dtype, void* stream);

/*
 * Mixture of experts; the routing never leaves the device.
 *   mv_moe_route    idx, weight (tokens, top): largest logits + bias, softmax over them (with over_all: over all
 *                   experts), times scale.  With `groups` > 1 the experts are that many equal runs, and only those of the
 *                   `keep` runs with the largest maxima can be chosen
 *   mv_moe_sort     stable sort of the tokens * top entries by expert: pos[entry] = row, row_token[row] = token,
 *                   offsets (experts + 1) = row ranges
 *   mv_gather_rows  out[r] = x[row_token[r]]
 *   mv_grouped_rows rows of expert e times w[e]^T (out_dim, in_dim); with an activation (enum mv_act) w[e] =
 *                   [gate; up] and the result is the gate applied to up
 * No counterpart in the reference.
 */
int mv_moe_route(int32_t* idx, float* weight, const float* logits, int64_t logits_stride, const
    float* bias, int64_t tokens, int experts, int top, int groups, int keep, int over_all, float scale, void* stream);
int64_t mv_moe_sort_workspace_bytes(int64_t tokens, int experts, int top);
int mv_moe_sort(int32_t* pos, int32_t* row_token, int32_t* offsets, const int32_t* idx, int64_t
    tokens, int experts, int top, void* workspace, int64_t workspace_bytes, void* stream);
int mv_gather_rows(void* out, const void* x, int64_t x_stride, const int32_t* row_token, int64_t
    rows, int width, int dtype, void* stream);
int mv_grouped_rows(void* out, const void* x, const void* w, const int32_t* offsets, int experts,
    int64_t rows, int in_dim, int out_dim, int act, float limit, int dtype, void* stream);

/*
 * mv_grouped_rows on the tensor cores (tcgen05), bf16, in_dim a multiple of 8.  A bounded wait that runs out is
 * reported in *error_word, as by mv_prefill_varlen.
 */
int mv_grouped_gemm(void* out, const void* x, const void* w, const int32_t* offsets, int experts,
    int64_t rows, int in_dim, int out_dim, int act, float limit, int* error_word, void* stream);

/*
 * mv_latent_attention_rows for one query row per sequence on tensor cores, bf16: rank a multiple of 16 up to 512,
 * rank + rot_dim a multiple of 32 up to 576, at most 1,024 rows (workspace_bytes returns -1 otherwise), blocks of 8, 16,
 * 32 or a multiple of 64 tokens.  Cache rows must hold finite values.  Bounded waits report in *error_word.  Sequence b has
 * positions[b] + 1 keys; rows with active[b] < 0 (active may be null) have none and give zeros.
 */
int64_t mv_latent_decode_workspace_bytes(int batch, int heads, int rank, int rot_dim);
int mv_latent_decode(void* out, int64_t out_stride, int64_t out_head_stride, const void* q_lat,
    int64_t q_lat_stride, int64_t q_lat_head_stride, const void* q_rot, int64_t q_rot_stride,
    int64_t q_rot_head_stride, const void* cache, const int32_t* block_tables, int64_t bt_stride,
    int max_blocks, int block_size, int64_t num_blocks, const int64_t* positions, const int32_t*
    active, const void* sink, int batch, int heads, int rank, int rot_dim, float scale, void*
    workspace, int64_t workspace_bytes, int* error_word, void* stream);

/*
 * Prefill of latent attention with keys and values expanded per head, bf16, tcgen05.
 *   mv_latent_gather   out[cu_k[s] + j] = cache row of position first[s] + j of sequence s (first null: j; bf16 or fp32,
 *                      rows of whole 16 bytes)
 *   mv_latent_prefill  q (tokens, heads * (dim + rot_dim)), k (keys, heads * dim), k_rot (keys, rot_dim) shared by the
 *                      heads, v (keys, heads * vdim); row strides in elements; sequence s has queries cu_q[s] .. at the
 *                      end of its keys cu_k[s] ..; sizes multiples of 8, 64-column boxes: at most three for dim and
 *                      rot_dim together, two for vdim; sink may be null.  Bounded waits report in *error_word.
 */
int mv_latent_gather(void* out, const void* cache, const int32_t* cu_k, const int32_t* first, int
    num_seqs, int64_t keys, const int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size, int64_t
    num_blocks, int row, int dtype, void* stream);
int mv_latent_prefill(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* k,
    int64_t k_stride, const void* k_rot, int64_t k_rot_stride, const void* v, int64_t v_stride,
    const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int64_t tokens, int64_t keys, int heads,
    int dim, int rot_dim, int vdim, float scale, const void* sink, int* error_word, void* stream);

/*
 * mv_ssm_scan in chunks of 64 tokens on tensor cores, bf16; every sequence of cu must be a portion.  `takes` tells
 * whether the sizes are supported (state 32, 64 or 128, vdim a multiple of 8).
 */
int mv_ssm_chunk_takes(int vdim, int state_dim);
int mv_ssm_chunk_scan(void* y, int64_t y_stride, const void* xbc, int64_t xbc_stride, const void*
    dt, int64_t dt_stride, const void* dt_bias, const void* A_log, const void* D, const int32_t* cu,
    int num_seqs, const int32_t* slots, const int32_t* start, float* state, int num_slots, int
    heads, int vdim, int state_dim, int groups, void* stream);

/*
 * One token per sequence, convolution included: u holds the rows before it, conv_state is read only (advance it with
 * mv_conv_state_update afterwards); state as in mv_ssm_scan.  vdim and state_dim multiples of 4.
 */
int mv_ssm_step(void* y, const void* u, int64_t u_stride, const void* w, const void* bias, int taps,
    const void* conv_state, const void* dt, int64_t dt_stride, const void* dt_bias, const void*
    A_log, const void* D, int num_seqs, const int32_t* slots, const int32_t* start, float* state,
    int num_slots, int heads, int vdim, int state_dim, int groups, int dtype, void* stream);

/*
 * Grouped-query attention with a sliding window over a paged cache of rows [kv_heads * dim keys | kv_heads * vdim
 * values].  Position i sees the keys j with 0 <= i - j < window; score = scale (q . k) + bias[h * bias_stride +
 * min(i - j, distances - 1)] (fp32; null: none); exp(sink[h]) joins the denominator (null: none).
 *   mv_kv_norm_store          q (in place) and k, each row of all heads: RMS norm with a weight per row; [k | v] goes to
 *                             kv_out (tokens, row; may be null) and to cache[slot] (slot < 0 skips)
 *   mv_window_attention_rows  any sizes up to vdim 1,024; token t belongs to the sequence of cu_q (null: row t)
 *   mv_window_decode          one token per sequence, bf16, dim and vdim multiples of 8 up to 256; workspace_bytes is
 *                             -1 when the sizes are not taken, most_keys = min(window, max_blocks * block_size)
 *   mv_window_prefill         packed queries and keys as in mv_latent_prefill (a sequence's keys begin at or before the
 *                             first one that its first query sees), bf16, dim up to 192, vdim up to 128, multiples of 8;
 *                             mv_window_prefill_distances = largest `distances` taken (-1: sizes not taken)
 *   mv_qkv_rope_store         q (in place) and k: RMS norm per head with a weight (dim), then pairs of neighbouring columns
 *                             2i, 2i + 1 of the first `dims` turned by the angle in row positions[t], column i of cos_t and
 *                             sin_t (table_rows, dims / 2); q of head h times temp[h] (null: 1).  v: its pairs turned by
 *                             vcos_t, vsin_t (table_rows, vdim / 2; null: as it is).  [k: kv_heads * dim | v: v_heads *
 *                             vdim] goes to kv_out and cache as above; kv_heads and v_heads 0: queries only; heads 0: keys and
 *                             values only; k_weight null: keys without a norm.  dim and vdim up to 1,024
 * turn (vdim / 2, table_rows, 2) of the attention entries: the result of position i is turned in the same pairs by the
 * opposite of the angles whose (cos, sin) are at [pair, i] (null: not).  out is (tokens, heads * vdim).  No counterpart in the reference.
 */
int mv_kv_norm_store(void* q, const void* k, const void* v, int64_t stride, const void* q_weight, const
    void* k_weight, void* kv_out, void* cache, const int64_t* slot_mapping, int64_t num_slots, int64_t
    tokens, int q_rows, int k_rows, int v_rows, float eps, int dtype, void* stream);
int mv_qkv_rope_store(void* q, const void* k, const void* v, int64_t stride, const void* q_weight, const
    void* k_weight, const void* temp, const float* cos_t, const float* sin_t, int dims, const float*
    vcos_t, const float* vsin_t, int64_t table_rows, const int64_t* positions, void* kv_out, void* cache,
    const int64_t* slot_mapping, int64_t num_slots, int64_t tokens, int heads, int kv_heads, int v_heads, int dim,
    int vdim, float eps, int dtype, void* stream);
int mv_window_attention_rows(void* out, const void* q, int64_t q_stride, const void* cache, const
    int32_t* block_tables, int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks,
    const int32_t* cu_q, int num_seqs, const int64_t* positions, const float* bias, int64_t
    bias_stride, int distances, const void* sink, const float* turn, int64_t table_rows, int64_t tokens, int heads, int kv_heads, int dim, int vdim, int64_t window, float
    scale, int dtype, void* stream);
int64_t mv_window_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, int64_t
    most_keys);
int mv_window_decode(void* out, const void* q, int64_t q_stride, const void* cache, const int32_t*
    block_tables, int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int64_t*
    positions, const float* bias, int64_t bias_stride, int distances, const void* sink, const float*
    turn, int64_t table_rows, int batch, int heads, int kv_heads, int dim, int vdim,
    int64_t window, float scale, void* workspace, int64_t workspace_bytes, void* stream);
int mv_window_prefill_distances(int dim, int vdim);
int mv_window_prefill(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* k,
    int64_t k_stride, const void* v, int64_t v_stride, const int32_t* cu_q, const int32_t* cu_k, int
    num_seqs, int64_t tokens, int64_t keys, int heads, int kv_heads, int dim, int vdim, int64_t window,
    float scale, const float* bias, int64_t bias_stride, int distances, const void* sink, const float*
    turn, int64_t table_rows, const int64_t* positions, int* error_word, void* stream);

/*
 * Matrix-state recurrences, fp32 state (num_slots, heads, dim, vdim) updated in place, one read-out per token; dim up
 * to 256.  cu, slots and start as in mv_conv_silu.  With cu null (one token per sequence) the head's norm and the output
 * gate follow in the same launch: out = rms_norm(o) * norm_w * silu(gate), norm_w (vdim); with cu they are ignored.
 *   mv_gla_scan    S <- diag(sigmoid(z)^(1 / tau)) S + k v^T,  o = S^T (q_scale q);  rows of q, k, v share one stride
 *   mv_delta_scan  S <- g S;  u = sigmoid(beta) (v - S^T k);  S <- S + k u^T;  o = S^T q, with q and k scaled to unit
 *                  length per head (1e-6 added to the sum of squares), q by q_scale too, and
 *                  g = exp(-exp(A_log) softplus(a + dt_bias)); rows of qkv are [q: kv_heads * dim | k | v: heads * vdim],
 *                  after the convolution and silu, or with cu null before them (conv_state is read only)
 * dtype MV_BF16 or MV_F32.  No counterpart in the reference.
 */
int mv_gla_scan(void* out, int64_t out_stride, const void* q, const void* k, const void* v, int64_t
    stride, const void* z, int64_t z_stride, float tau, const int32_t* cu, int num_seqs, const
    int32_t* slots, const int32_t* start, float* state, int num_slots, int heads, int dim, int vdim,
    float q_scale, const void* gate, int64_t gate_stride, const void* norm_w, float eps, int dtype,
    void* stream);
int mv_delta_scan(void* out, int64_t out_stride, const void* qkv, int64_t stride, const void* beta,
    const void* a, int64_t ba_stride, const void* A_log, const void* dt_bias, const int32_t* cu, int
    num_seqs, const int32_t* slots, const int32_t* start, float* state, int num_slots, int heads,
    int kv_heads, int dim, int vdim, float q_scale, const void* conv_w, int taps, const void*
    conv_state, const void* gate, int64_t gate_stride, const void* norm_w, float eps, int dtype,
    void* stream);

/*
 * The same recurrences for packed portions in chunks of 64 tokens on tensor cores, bf16: dim a multiple of 8 up to 128,
 * vdim a multiple of 8, rows on 16-byte boundaries.  tokens = cu[num_seqs]; workspace_bytes is -1 when the sizes are not
 * taken.
 */
int64_t mv_gla_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim);
int mv_gla_chunk_scan(void* out, int64_t out_stride, const void* q, const void* k, const void* v,
    int64_t stride, const void* z, int64_t z_stride, float tau, const int32_t* cu, int num_seqs,
    int64_t tokens, const int32_t* slots, const int32_t* start, float* state, int num_slots, int
    heads, int dim, int vdim, float q_scale, void* workspace, int64_t workspace_bytes, void* stream);
int64_t mv_delta_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim);
int mv_delta_chunk_scan(void* out, int64_t out_stride, const void* qkv, int64_t stride, const void*
    beta, const void* a, int64_t ba_stride, const void* A_log, const void* dt_bias, const int32_t* cu,
    int num_seqs, int64_t tokens, const int32_t* slots, const int32_t* start, float* state, int
    num_slots, int heads, int kv_heads, int dim, int vdim, float q_scale, void* workspace, int64_t
    workspace_bytes, void* stream);

/*
 * Matrix memory with exponential gates and a running maximum (mLSTM), fp32 state S (num_slots, heads, dim, vdim), n (num_slots,
 * heads, dim), m (num_slots, heads), updated in place; cu, slots and start as in mv_conv_silu.  Per head and token, with
 * i = cap tanh((zi + i_b) / cap), f = logsigmoid(cap tanh((zf + f_b) / cap)):
 *   m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k;  m <- m'
 *   o = S^T q / (max(|n . q|, exp(-m)) + 1e-6), q scaled by q_scale
 * gates (tokens, 2 * heads) fp32 holds [zi | zf], rows of q, k, v share one stride; dim up to 256.
 *   mv_mlstm_gates       portions: chain (tokens, heads, 4) = i, f, m before and after the token; m advances
 *   mv_mlstm_scan        portions, token by token: out = S^T q, den (tokens, heads) fp32 = its denominator
 *   mv_mlstm_chunk_scan  the same in chunks of 64 tokens on tensor cores, bf16: dim a multiple of 8 up to 128, vdim a multiple
 *                        of 8, rows on 16-byte boundaries; tokens = cu[num_seqs]; workspace_bytes is -1 when the sizes are
 *                        not taken
 *   mv_mlstm_step        one token per sequence: out = rms_norm(o) * norm_w * sigmoid(gate), norm_w (heads * vdim); the gates'
 *                        logits are x (tokens, width) times gates_w (2 * heads, width)
 * dtype MV_BF16 or MV_F32.  No counterpart in the reference.
 */
int mv_mlstm_gates(float* chain, const float* gates, int64_t gates_stride, const void* i_b, const void* f_b,
    float cap, const int32_t* cu, int num_seqs, const int32_t* slots, const int32_t* start, float* m_state,
    int num_slots, int heads, int dtype, void* stream);
int mv_mlstm_scan(void* out, int64_t out_stride, float* den, const void* q, const void* k, const void* v,
    int64_t stride, const float* chain, const int32_t* cu, int num_seqs, const int32_t* slots, const
    int32_t* start, float* S, float* n, int num_slots, int heads, int dim, int vdim, float q_scale, int
    dtype, void* stream);
int64_t mv_mlstm_chunk_workspace_bytes(int64_t tokens, int num_seqs, int heads, int dim, int vdim);
int mv_mlstm_chunk_scan(void* out, int64_t out_stride, float* den, const void* q, const void* k, const void*
    v, int64_t stride, const float* chain, const int32_t* cu, int num_seqs, int64_t tokens, const int32_t*
    slots, const int32_t* start, float* S, float* n, int num_slots, int heads, int dim, int vdim, float
    q_scale, void* workspace, int64_t workspace_bytes, void* stream);
int mv_mlstm_step(void* out, int64_t out_stride, const void* q, const void* k, const void* v, int64_t stride,
    const void* x, int64_t x_stride, const void* gates_w, int width, const void* i_b, const void* f_b, float
    cap, int num_seqs, const int32_t* slots, const int32_t* start, float* S, float* n, float* m, int num_slots, int heads, int
    dim, int vdim, float q_scale, const void* gate, int64_t gate_stride, const void* norm_w, float eps, int
    dtype, void* stream);

/*
 * Between two sublayers of a decoder with several residual streams x (rows, streams, width) fp32, at most 16.  The new streams
 * x_t = sum_s mix[s, t] x_s + w_out[t] y (all from the old ones; with ids: every stream = the embedding row), then
 * u = sum_s w_in[s] x_s (null: plain sum) and h = layer norm of u with norm_w and norm_b (norm_b null: RMS norm).
 * Rows below conv_rows are one-token sequences with slots and starts as in mv_conv_silu: with taps > 0, out = h + causal
 * convolution of h with taps_t (taps, width), whose inputs conv_state (num_slots, taps - 1, width) keeps and which moves on.
 * Without taps out = h.  The h of the other rows goes to raw, from its first row on.  dtype MV_BF16 or MV_F32 of all but x.
 * No counterpart in the reference.
 */
int mv_stream_step(void* out, void* raw, float* x, const int64_t* ids, const void* embed, int64_t vocab, const
    void* y, int64_t y_stride, const void* mix, const void* w_out, const void* w_in, const void* norm_w,
    const void* norm_b, const void* taps_t, int taps, void* conv_state, const int32_t* slots, const int32_t*
    start, int num_slots, int64_t conv_rows, int64_t rows, int width, int streams, float eps, int dtype,
    void* stream);

/*
 * Grouped-query attention whose softmax weights are mixed across the heads, over the same kind of cache (key and value rows of
 * kv_heads heads each), causal:
 *   s = cap tanh(scale (q . k) / cap) - r1[h] ln(1 + r2[h] (i - j)),  w = softmax over j <= i,
 *   w'_h = sum_g talk[h, g] w_g,  out_h = out_scale sum_j w'_h(j) v_j of h's own value head
 * r1, r2 (heads) and talk (heads, heads) fp32.
 *   mv_talk_decode          one token per sequence, bf16, dim and vdim multiples of 8 up to 256, cap up to 60; workspace_bytes is
 *                           -1 when sizes or cap are not taken, most_keys = max_blocks * block_size
 *   mv_talk_prefill         packed queries, keys and values (row strides in elements) as in mv_window_prefill, bf16, dim up to
 *                           128, vdim up to 256, multiples of 8, cap up to 60 (mv_talk_prefill_takes): a (tokens, heads,
 *                           kv_heads, vdim) = every head's w over the values of every value head
 *   mv_talk_attention_rows  any sizes, a as above in fp32; cu_q as in mv_window_attention_rows
 *   mv_head_mix             out_h = out_scale sum_g talk[h, g] a[g, value head of h]; a in fp32 or in the type of out
 * No counterpart in the reference.
 */
int64_t mv_talk_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, float cap, int64_t most_keys);
int mv_talk_decode(void* out, int64_t out_stride, const void* q, int64_t q_stride, const void* cache, const int32_t*
    block_tables, int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int64_t* positions,
    const float* r1, const float* r2, const float* talk, float cap, int batch, int heads, int kv_heads, int dim, int
    vdim, float scale, float out_scale, void* workspace, int64_t workspace_bytes, void* stream);
int mv_talk_prefill_takes(int dim, int vdim, float cap);
int mv_talk_prefill(void* a, const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t
    v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int64_t tokens, int64_t keys, const float* r1,
    const float* r2, float cap, int heads, int kv_heads, int dim, int vdim, float scale, int* error_word, void* stream);
int mv_talk_attention_rows(float* a, const void* q, int64_t q_stride, const void* cache, const int32_t* block_tables,
    int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int32_t* cu_q, int num_seqs, const
    int64_t* positions, const float* r1, const float* r2, float cap, int64_t tokens, int heads, int kv_heads, int dim,
    int vdim, float scale, int dtype, void* stream);
int mv_head_mix(void* out, int64_t out_stride, const void* a, int a_dtype, const float* talk, float out_scale, int64_t
    tokens, int heads, int kv_heads, int vdim, int dtype, void* stream);

/*
 * Differential attention in chunks: a head has two maps, with queries (heads, 2, dim) and keys (kv_heads, 2, dim) of their own
 * and the same values; position i sees j <= i with floor(j / chunk) = floor(i / chunk).  Cache rows are [kv_heads * 2 * dim keys
 * | kv_heads * vdim values].  out = rms_norm(a1 - lambda a2) mult sigmoid(gate), the norm over the head's vdim, without weight.
 *   mv_diff_decode          one token per sequence, bf16, dim up to 128, vdim up to 256, multiples of 8; workspace_bytes is -1
 *                           when the sizes are not taken, most_keys = min(chunk, max_blocks * block_size)
 *   mv_diff_prefill         packed rows; a sequence's keys begin at the beginning of a chunk; scale > 0; bf16, dim and vdim up to
 *                           128, multiples of 8 (mv_diff_prefill_takes)
 *   mv_diff_attention_rows  any sizes: a (tokens, heads, 2, vdim) = a1 and a2 in fp32
 *   mv_diff_norm_gate       the rest of it, from a
 * No counterpart in the reference.
 */
int64_t mv_diff_decode_workspace_bytes(int batch, int heads, int kv_heads, int dim, int vdim, int64_t most_keys);
int mv_diff_decode(void* out, const void* q, int64_t q_stride, const void* cache, const int32_t* block_tables, int64_t
    bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int64_t* positions, int64_t chunk, const void*
    gate, int64_t gate_stride, float lambda, float mult, float eps, int batch, int heads, int kv_heads, int dim, int
    vdim, float scale, void* workspace, int64_t workspace_bytes, void* stream);
int mv_diff_prefill_takes(int dim, int vdim);
int mv_diff_prefill(void* out, const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t
    v_stride, const int32_t* cu_q, const int32_t* cu_k, int num_seqs, int64_t tokens, int64_t keys, int64_t chunk,
    const void* gate, int64_t gate_stride, float lambda, float mult, float eps, int heads, int kv_heads,
    int dim, int vdim, float scale, int* error_word, void* stream);
int mv_diff_attention_rows(float* a, const void* q, int64_t q_stride, const void* cache, const int32_t* block_tables,
    int64_t bt_stride, int max_blocks, int block_size, int64_t num_blocks, const int32_t* cu_q, int num_seqs, const
    int64_t* positions, int64_t chunk, int64_t tokens, int heads, int kv_heads, int dim, int vdim, float scale, int
    dtype, void* stream);
int mv_diff_norm_gate(void* out, const float* a, const void* gate, int64_t gate_stride, float lambda, float mult, float
    eps, int64_t tokens, int heads, int vdim, int dtype, void* stream);

/*
 * Time mixing on a matrix state: o = (S + diag(bonus) k v^T)^T r, then S <- diag(exp(-exp(z + w0))) S + k v^T; z (tokens, heads *
 * dim) fp32, w0 and bonus (heads, dim); state, cu, slots and start as in mv_gla_scan.  With cu null the norm and the gate follow:
 * out = rms_norm(o) * norm_w * silu(gate) * out_scale, norm_w (heads * vdim).  mv_time_chunk_scan: portions in chunks of 64 tokens
 * on tensor cores, with the sizes and the workspace of mv_gla_chunk_scan.  No counterpart in the reference.
 */
int mv_time_scan(void* out, int64_t out_stride, const void* r, const void* k, const void* v, int64_t stride, const float*
    z, int64_t z_stride, const void* w0, const void* bonus, const int32_t* cu, int num_seqs, const int32_t* slots, const
    int32_t* start, float* state, int num_slots, int heads, int dim, int vdim, const void* gate, int64_t gate_stride,
    const void* norm_w, float eps, float out_scale, int dtype, void* stream);
int mv_time_chunk_scan(void* out, int64_t out_stride, const void* r, const void* k, const void* v, int64_t stride, const
    float* z, int64_t z_stride, const void* w0, const void* bonus, const int32_t* cu, int num_seqs, int64_t tokens, const
    int32_t* slots, const int32_t* start, float* state, int num_slots, int heads, int dim, int vdim, void* workspace,
    int64_t workspace_bytes, void* stream);

/*
 * Between two sublayers of a decoder with one fp32 residual stream and an element-wise norm: out = tanh(alpha x') w + b, where
 * x_out = x' is x_in plus y (rows, y_stride), or plus sum_k top_weights[t, k] y[pos[t, k]] (pos not null), or with ids the
 * embedding row, to which sin(position inv_freq[i]) and cos of the same are added in columns 2i and 2i + 1 (inv_freq null: not).
 * mixes > 0: mixed[m] (rows, width) = out + (before - out) mu[m], with the out of the sequence's token before (zeros for its
 * first); kept (num_slots, width) holds the last one.  A sequence with one row in this step moves its kept row on; for longer
 * ones mv_conv_state_update does it afterwards.  With mixes x_out and x_in must differ.  cu, slots and start as in mv_conv_silu.
 *   mv_xielu      out = a z^2 + z / 2 for z > 0, else b (e^z - 1 - z) + z / 2
 *   mv_tanh_rows  out = tanh(y), y in fp32
 * dtype MV_BF16 or MV_F32 of all but x, y of mv_tanh_rows and top_weights.  No counterpart in the reference.
 */
int mv_tanh_step(void* out, float* x_out, const float* x_in, const int64_t* ids, const void* embed, int64_t vocab, const
    int64_t* positions, const double* inv_freq, const void* y, int64_t y_stride, const int32_t* pos, const float*
    top_weights, int top, float alpha, const void* w, const void* b, void* mixed, const void* mu, int mixes, void* kept,
    const int32_t* slots, const int32_t* start, int num_slots, const int32_t* cu, int num_seqs, int64_t rows, int width,
    int dtype, void* stream);
int mv_xielu(void* out, const void* y, int64_t y_stride, float a, float b, int64_t rows, int cols, int dtype, void* stream);
int mv_tanh_rows(void* out, const float* y, int64_t y_stride, int64_t rows, int cols, int dtype, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* MINIVLLM_B200_H */
