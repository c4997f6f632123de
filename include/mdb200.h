/*
 * libmdb200 -- C ABI of the B200 (sm_100a) block-diffusion decode kernels.
 *
 * Every entry point takes plain device pointers, sizes and a CUDA stream
 * (cudaStream_t passed as void*); nothing here names a torch type.  All
 * buffers are owned by the caller.  Calls are asynchronous on `stream`, do
 * not allocate and do not synchronise unless stated.  The return value is
 * MDB_OK or a negative MDB_ERR_* detected on the host before any launch.
 * Conditions only the device can see (a cache slot outside the pool, a
 * bounded wait that ran out) set a bit in a device status word instead of
 * trapping; read it with mdb_last_device_status().
 *
 * Paths in the comments are relative to the reference project root; NV/
 * abbreviates engines/nano_dvlm/nanovllm/.  bf16 means __nv_bfloat16.
 */
#ifndef MDB200_H
#define MDB200_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef void* mdb_stream_t; /* cudaStream_t */

enum {
  MDB_OK = 0,
  MDB_ERR_ARG = -1,         /* null pointer, non-positive size, inconsistent dims */
  MDB_ERR_ALIGN = -2,       /* pointer or stride not 16-byte aligned */
  MDB_ERR_UNSUPPORTED = -3, /* shape outside what the kernels are built for */
  MDB_ERR_CUDA = -4,        /* the launch itself was refused by the runtime */
  MDB_ERR_WORKSPACE = -5,   /* workspace smaller than *_workspace_bytes() */
  MDB_ERR_STATIC_LIMIT = -6 /* request needs more than the fixed scratch of an allocation-free entry point */
};

/* bits of the device status word */
enum {
  MDB_STATUS_BAD_SLOT = 1u,     /* slot_mapping entry outside [0, num_slots) and not -1: row skipped */
  MDB_STATUS_BAD_PAGE = 2u,     /* page-table entry outside [0, num_pages) (page 0 is read in its place) or a context
                                   longer than the page-table row can address (cut to the row): output rows invalid */
  MDB_STATUS_BAD_TOKEN = 4u,    /* token id outside the embedding table: row zeroed */
  MDB_STATUS_BAD_POSITION = 8u, /* position outside the rotary table: row left unrotated */
  MDB_STATUS_WAIT_TIMEOUT = 16u, /* a bounded wait on a peer flag or barrier expired */
  MDB_STATUS_LAYOUT = 32u        /* a kernel found its shared memory placed otherwise than it was built for and did nothing */
};

const char* mdb_strerror(int code);
int mdb_version(void);

/* Process-wide switches (no counterpart in the reference; for measurement and
 * fault isolation).  MDB_OPT_PDL: 1 = kernels are chained with programmatic
 * dependent launch (default), 0 = plain stream order.  MDB_OPT_GEMM_PAIR: GEMMs
 * of many rows on pairs of CTAs (tcgen05.mma.cta_group::2, tiles of 256 x 256):
 * 1 = from 2048 rows (default), 2 = from 256 rows, 0 = never.
 * MDB_OPT_WAIT_LIMIT_US: how long a wait inside a kernel (mbarrier, peer flag)
 * may last before it gives up and raises MDB_STATUS_WAIT_TIMEOUT, in
 * microseconds (default 2 000 000); written to the current device, blocking. */
enum { MDB_OPT_PDL = 1, MDB_OPT_GEMM_PAIR = 3, MDB_OPT_WAIT_LIMIT_US = 4 };
int mdb_set_option(int option, int value);
/* Measurement aid: registers a device buffer (uint64 count, then (kernel,
 * event, globaltimer ns) triples) that block 0 of the traced kernels appends
 * to; NULL switches tracing off.  The stamps exist only in a library built
 * with -DMDB_TRACE (MDB_TRACE=1 python mineru-diffusion_b200/build.py); in the
 * normal build the call registers the buffer and nothing is ever written to
 * it: even testing the buffer pointer in the kernels costs 7 % of a short step. */
int mdb_set_trace(void* buffer, int64_t bytes);
int mdb_get_option(int option);

/* Copies the status word of the current device to *out (host memory) after
 * synchronising the device; clear != 0 resets it.  Plays the part of the
 * reference's host asserts (NV/layers/attention.py:36-39). */
int mdb_last_device_status(unsigned int* out, int clear);

/* ---- paged KV write/commit --------------------------------------------- */

/* Replaces store_kvcache / store_kvcache_kernel (NV/layers/attention.py:10-40).
 * Row i of key/value (row_elems = Hkv*D bf16, row strides in elements) is
 * copied to k_cache/v_cache row slot_mapping[i]; slot -1 skips the row. */
int mdb_kv_commit(const void* key, int64_t key_stride, const void* value, int64_t value_stride, void* k_cache,
                  void* v_cache, const int32_t* slot_mapping, int n_tokens, int row_elems, int64_t num_slots,
                  mdb_stream_t stream);

/* ---- block attention over the paged cache (decode / denoise step) -------- */

/* Replaces flash_attn_with_kvcache(q, k_cache, v_cache, cache_seqlens,
 * block_table, softmax_scale, causal=False) as called at
 * NV/layers/sdar_attention.py:50-55.  q/out: [bs, block, hq, 128] bf16;
 * caches: [num_pages, 256, hkv, 128] bf16; block_table: [bs, table_stride]
 * int32 (-1 padded); ctx_lens: [bs] int32, 0 makes the request a no-op (its
 * output rows are zeroed).  Every query row sees keys [0, ctx).  The key range
 * of each request is cut into at most nsplit parts processed by different
 * CTAs (equal shares of its context, rounded up to whole key tiles and never
 * shorter than 256 keys, so a short context uses fewer parts than asked for);
 * nsplit > 1 needs the workspace. */
int64_t mdb_attn_paged_workspace_bytes(int bs, int block, int hq, int nsplit);
int mdb_attn_block_paged(const void* q, const void* k_cache, const void* v_cache, void* out,
                         const int32_t* block_table, int table_stride, const int32_t* ctx_lens, int bs, int block,
                         int hq, int hkv, int num_pages, float softmax_scale, int nsplit, void* workspace,
                         int64_t workspace_bytes, mdb_stream_t stream);

/* No counterpart in the reference.  Same operation and arguments as
 * mdb_attn_block_paged, but without a workspace argument: the split partials
 * go to a fixed 8 MiB array that lives inside the library (one per device,
 * held from load to exit), and the call allocates nothing.  It is meant for
 * hosts that cannot provide scratch memory, e.g. an engine whose KV-cache
 * pool has taken all remaining device memory, or a serving thread that must
 * not enter the allocator.  A request whose partials would not fit
 * (mdb_attn_paged_workspace_bytes(bs, block, hq, nsplit) above
 * mdb_attn_block_paged_noalloc_limit()) is refused with MDB_ERR_STATIC_LIMIT;
 * lower nsplit or bs.  The first call on each device resolves the array's
 * device address and should be made outside stream capture.  Calls share the
 * array: calls that overlap on the GPU race, so issue them on one stream. */
int64_t mdb_attn_block_paged_noalloc_limit(void);
int mdb_attn_block_paged_noalloc(const void* q, const void* k_cache, const void* v_cache, void* out,
                                 const int32_t* block_table, int table_stride, const int32_t* ctx_lens, int bs,
                                 int block, int hq, int hkv, int num_pages, float softmax_scale, int nsplit,
                                 mdb_stream_t stream);

/* ---- staircase (block-causal, right-aligned) prefill attention ----------- */

/* Replaces sparse_attn_varlen(q, k, v, cu_seqlens_q, cu_seqlens_k,
 * staircase_size) (NV/kernels/triton/attention/block_prefill_attention_v2.py:
 * 17-202, call site NV/layers/sdar_attention.py:39-47).  Packed sequences:
 * q/out rows of hq*128, k/v rows of hkv*128, row strides in elements;
 * cu_seqlens: [nseq+1] int32 (queries and keys share it: self-attention).
 * Query i of a T-token sequence sees keys j <= ((i+pad)/S+1)*S-1-pad with
 * pad = ceil(T/S)*S - T.  stairs must be a power of two in [1,128].
 * total_tokens = cu_seqlens[nseq] = the row count of q, k, v and out (the host
 * knows it; the TMA descriptors of the tcgen05 kernel are bounded by it). */
int mdb_attn_staircase_varlen(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v,
                              int64_t v_stride, void* out, int64_t out_stride, const int32_t* cu_seqlens, int nseq,
                              int max_seqlen, int64_t total_tokens, int hq, int hkv, int stairs, mdb_stream_t stream);

/* ---- linear layers -------------------------------------------------------- */

/* In every entry of this section w is model data: with MDB_OPT_PDL on, a kernel
 * requests its first weight tiles while the preceding kernel of the stream may
 * still be running (weights are the only operand fetched that early), so w must
 * not be something a library call issued just before on the same stream writes.
 * Activations, outputs and workspaces carry the usual stream order. */

/* y[m,n] = x[m,k] * w[n,k]^T, bf16 in, fp32 accumulate, bf16 out: F.linear as
 * used by NV/layers/linear.py:72-73,153-154 and NV/layers/embed_head.py:67.
 * m <= 64 with n % 128 == 0 streams the weight once; everything else runs the
 * tcgen05 tile kernel (clusters of CTAs split k when the tiles are few, pairs
 * of CTAs share a tile from 2048 rows on); k % 64 == 0 and n % 8 == 0. */
int mdb_gemm_bf16(const void* x, int64_t ldx, const void* w, void* y, int64_t ldy, int m, int n, int k,
                  mdb_stream_t stream);

/* Same product for m <= 256 as a weight-streaming kernel that cuts k into
 * ksplit slices and writes fp32 partial sums partials[ksplit][m][n]; the
 * consumers below add the slices in index order, round to bf16 where F.linear
 * would, and apply the layer that follows.  (n % 128 == 0, k % 64 == 0, no
 * empty slice; the tensor-parallel form below takes m <= 64.) */
int mdb_gemm_pick_ksplit(int m, int n, int k); /* a ksplit that suits the kernel these shapes will run on */
int64_t mdb_gemm_splitk_workspace_bytes(int m, int n, int ksplit);
int mdb_gemm_splitk_partials(const void* x, int64_t ldx, const void* w, float* partials, int m, int n, int k,
                             int ksplit, mdb_stream_t stream);

/* gate_up projection fused with SiLU*mul (NV/models/sdar.py:109-111,
 * NV/layers/activation.py:12-15): w is [2*inter, k] with gate rows first;
 * act[m, inter] = bf16(silu_fp32(bf16(gate))) * bf16(up).  m <= 64 streams the
 * weight once (inter % 64 == 0, k % 64 == 0); larger m runs the tcgen05 tile
 * kernel (inter % 128 == 0, k % 64 == 0). */
int mdb_gemm_gateup_swiglu(const void* x, int64_t ldx, const void* w_gate_up, void* act, int64_t ld_act, int m,
                           int inter, int k, mdb_stream_t stream);

/* SiLU*mul on a materialised [m, 2*inter] bf16 matrix (SiluAndMul.forward, NV/layers/activation.py:12-15). */
int mdb_silu_mul(const void* gate_up, int64_t ld_in, void* act, int64_t ld_act, int m, int inter,
                 mdb_stream_t stream);

/* ---- fused reductions / element-wise layers -------------------------------- */

/* RMSNorm with fused residual add (NV/layers/layernorm.py:16-40).  The input
 * row is either x (bf16 [m,h]) or, when partials != NULL, the bf16-rounded
 * sum of nparts fp32 slices [nparts][m][h].  residual_in == NULL selects the
 * no-residual form (residual_out, if given, receives the input row). */
int mdb_add_rmsnorm(const void* x, const float* partials, int nparts, const void* residual_in, const void* weight,
                    float eps, void* y_out, void* residual_out, int m, int h, mdb_stream_t stream);

/* What follows qkv_proj in SDARAttention.forward (NV/models/sdar.py:73-82):
 * split q|k|v, per-head RMSNorm of q and k, NeoX rotary embedding from the
 * fp32 cos|sin table (NV/layers/rotary_embedding.py:6-48), then the KV store
 * of Attention.forward (NV/layers/sdar_attention.py:37-38).  Input row is
 * qkv (bf16 [m, (hq+2hkv)*128], row stride ld_qkv) or fp32 partials as above.
 * q_out [m, hq*128]; k_out/v_out [m, hkv*128] optional (prefill needs them
 * contiguous); slot_mapping optional (NULL: no cache write). */
int mdb_qknorm_rope_commit(const void* qkv, int64_t ld_qkv, const float* partials, int nparts,
                           const int64_t* positions, const float* rope_table, int max_pos, const void* q_norm_w,
                           const void* k_norm_w, float eps, const int32_t* slot_mapping, void* q_out, void* k_out,
                           void* v_out, void* k_cache, void* v_cache, int64_t num_slots, int m, int hq, int hkv,
                           mdb_stream_t stream);

/* qkv_proj and everything mdb_qknorm_rope_commit does, in one kernel for many
 * rows (prefill, batched decode): y = x w_qkv^T on the tcgen05 tile GEMM whose
 * epilogue rounds the projection to bf16, applies the per-head q/k RMSNorm and
 * the rotary embedding and stores q, k, v (NV/models/sdar.py:73-82,
 * NV/layers/sdar_attention.py:37-38) -- the [m, (hq+2hkv)*128] projection
 * never reaches memory.  x bf16 [m,k] (row stride ldx), w_qkv bf16
 * [(hq+2hkv)*128, k]; other arguments as mdb_qknorm_rope_commit.
 * MDB_ERR_UNSUPPORTED unless k % 64 == 0 and ldx % 8 == 0. */
int mdb_gemm_qkv_rope_commit(const void* x, int64_t ldx, const void* w_qkv, int m, int k, const int64_t* positions,
                             const float* rope_table, int max_pos, const void* q_norm_w, const void* k_norm_w,
                             float eps, const int32_t* slot_mapping, void* q_out, void* k_out, void* v_out,
                             void* k_cache, void* v_cache, int64_t num_slots, int hq, int hkv, mdb_stream_t stream);

/* Row gather: out[i,:] = table[ids[i],:] (F.embedding at
 * NV/layers/embed_head.py:38; also the last-block row pick of the LM head at
 * NV/layers/embed_head.py:63-66). */
int mdb_gather_rows(const void* table, int64_t num_rows, const int64_t* ids, void* out, int m, int h,
                    mdb_stream_t stream);

/* ---- LM head + sampler ------------------------------------------------------ */

/* Replaces ParallelLMHead.forward + Sampler.prepare (NV/layers/embed_head.py:
 * 61-72, NV/layers/sampler.py:11-22) without materialising logits: for each of
 * the m rows, logit_v = bf16(hidden . w[v]) / T, x0 = argmax_v(logit_v +
 * noise_v) (lowest index wins a tie), conf = softmax(logit)[x0].
 * temperatures: [m / block] fp32, one per request.  noise_mode 0: none,
 * 1: `noise` points to fp32 [m, vocab] Gumbel values, 2: counter-based Gumbel
 * noise from (seed, step, row, column) -- mdb_gumbel_noise() writes out the
 * same values.  step_dev, if not NULL, points to a uint32 in device memory
 * that is added to `step` when the kernel runs, so a captured graph can be
 * replayed with fresh noise.  m <= 64 streams the weight once; larger m runs
 * the tile GEMM with the sampler reduction in its epilogue (an explicit noise
 * tensor with many rows goes through bf16 logits in the workspace). */
int64_t mdb_lmhead_workspace_bytes(int m, int vocab);
int mdb_lmhead_sample(const void* hidden, int64_t ld_hidden, const void* w, int m, int vocab, int h,
                      const float* temperatures, int block, int noise_mode, const float* noise, uint32_t seed,
                      uint32_t step, const uint32_t* step_dev, void* workspace, int64_t workspace_bytes,
                      int32_t* x0_out, float* conf_out, mdb_stream_t stream);

/* Same scan over already materialised bf16 logits [m, vocab] (row stride ld);
 * a workspace of mdb_lmhead_workspace_bytes(m, vocab) always suffices. */
int mdb_logits_sample(const void* logits, int64_t ld, int m, int vocab, const float* temperatures, int block,
                      int noise_mode, const float* noise, uint32_t seed, uint32_t step, const uint32_t* step_dev,
                      void* workspace, int64_t workspace_bytes, int32_t* x0_out, float* conf_out,
                      mdb_stream_t stream);

int mdb_gumbel_noise(float* out, int m, int vocab, uint32_t seed, uint32_t step, mdb_stream_t stream);

/* The unmask rule of Sampler.forward (NV/layers/sampler.py:28-54) on device:
 * per request, masked positions whose confidence is > threshold are replaced
 * by x0; if fewer than the request's quota qualify, the quota most confident
 * masked positions are taken instead (all of them when fewer are left; the
 * lowest index wins a tie).  quota = 1 is the nano engine's rule; the HF twin
 * takes its quota from a per-block schedule
 * (mineru_diffusion/modeling_mineru_diffusion.py:518-532,617-623): pass it per
 * request in quotas [bs] int32 (device; NULL: `quota` for every request).
 * block_ids [bs, block] int64 is updated in place; transfer_out [bs, block]
 * uint8; count_out [bs] int32 = positions unmasked.  Requests with no masked
 * position are left untouched.  A quota of 0 (the schedule's entry when a block
 * has more steps than tokens) transfers only what passes the threshold.
 * status_out, if not NULL, is a device word that receives the device status
 * word as it stands when this kernel runs (the step's kernels before it have
 * finished), and the status word is cleared: the host reads the step's status
 * in the same copy as its results instead of synchronising for it. */
int mdb_unmask_decide(int64_t* block_ids, const int32_t* x0, const float* conf, int bs, int block, int64_t mask_id,
                      float threshold, int quota, const int32_t* quotas, uint8_t* transfer_out, int32_t* count_out,
                      uint32_t* status_out, mdb_stream_t stream);

/* ---- tensor-parallel pair (TP = 2) -------------------------------------------------- */

/* Replaces dist.all_reduce in RowParallelLinear.forward (NV/layers/linear.py:153-157),
 * the logits gather of ParallelLMHead (NV/layers/embed_head.py:68-71) and the
 * handle plumbing NCCL does for them.  Each rank holds half of the heads, MLP
 * columns and vocabulary tiles.  The o_proj / down_proj GEMM of a rank stores
 * its fp32 k-slices into its own slice buffer AND, over NVLink, into the
 * peer's (plain stores from the epilogue), then writes a sequence number into
 * its CTA's flag slot in the peer's memory.  The consumer (RMSNorm with
 * residual add) waits, bounded, for the peer's slots and sums rank 0's slices
 * then rank 1's, so both ranks obtain bit-identical rows.  Sequence number =
 * (*epoch) * 256 + tag; the host advances *epoch every step, tag (1..255) is
 * distinct per producing launch within a step. */

/* Device memory the peer may map: allocate, export a 64-byte handle, import the
 * peer's handle (in the other process), release/free at shutdown.  Called at
 * engine start only. */
int mdb_tp_alloc(int64_t bytes, void** out);
int mdb_tp_free(void* ptr);
int mdb_tp_export(void* ptr, void* handle_out64);
int mdb_tp_import(const void* handle64, void** peer_ptr_out);
int mdb_tp_release(void* peer_ptr);

/* mdb_gemm_splitk_partials whose slices also go to peer_partials (same layout,
 * peer memory) and that signals peer_flags[cta]; m <= 64, n % 128 == 0,
 * k % 64 == 0.  mdb_tp_grid_size gives the number of CTAs = flag slots used. */
int mdb_gemm_splitk_partials_tp(const void* x, int64_t ldx, const void* w, float* partials, float* peer_partials,
                                int m, int n, int k, int ksplit, uint32_t* peer_flags, uint32_t tag,
                                const uint32_t* epoch, mdb_stream_t stream);
int mdb_tp_grid_size(int m, int n, int k, int ksplit);

/* mdb_add_rmsnorm that first waits for wait_count flag slots written by the peer. */
int mdb_add_rmsnorm_tp(const void* x, const float* partials, int nparts, const void* residual_in, const void* weight,
                       float eps, void* y_out, void* residual_out, int m, int h, const uint32_t* wait_flags,
                       int wait_count, uint32_t tag, const uint32_t* epoch, mdb_stream_t stream);

/* The same exchange for steps of more than 64 rows (RowParallelLinear.forward +
 * dist.all_reduce, NV/layers/linear.py:153-157, on the tcgen05 tile GEMM):
 * mdb_gemm_bf16_tp stores every bf16 output tile into y and, with plain stores
 * over NVLink, into y_peer (the landing buffer in the peer's mdb_tp_alloc
 * memory, same leading dimension); each CTA then raises peer_flags[cta].
 * *grid_out = number of CTAs launched = flag slots the consumer has to wait
 * for (both ranks launch the same shape).  MDB_ERR_UNSUPPORTED unless m > 64
 * and the shape suits the tile kernel (k % 64 == 0, n % 8 == 0, ldy % 8 == 0).
 * mdb_add_rmsnorm_tp_rows waits for those slots and takes bf16(x + x_peer) as
 * its input row (x: this rank's output, x_peer: the local landing buffer the
 * peer wrote), which is what the all-reduce of two bf16 tensors yields. */
int mdb_gemm_bf16_tp(const void* x, int64_t ldx, const void* w, void* y, void* y_peer, int64_t ldy, int m, int n, int k,
                     uint32_t* peer_flags, uint32_t tag, const uint32_t* epoch, int* grid_out, mdb_stream_t stream);
int mdb_add_rmsnorm_tp_rows(const void* x, const void* x_peer, const void* residual_in, const void* weight, float eps,
                            void* y_out, void* residual_out, int m, int h, const uint32_t* wait_flags, int wait_count,
                            uint32_t tag, const uint32_t* epoch, mdb_stream_t stream);

/* mdb_lmhead_sample over the vocabulary tiles [tile_begin, tile_begin + tile_count)
 * (128 rows each) of the full weight; the per-tile records (20 bytes per step
 * row) are mirrored into the peer's workspace instead of gathering logits, and
 * the merge waits for the peer's records. */
int mdb_lmhead_sample_tp(const void* hidden, int64_t ld_hidden, const void* w, int m, int vocab, int h,
                         const float* temperatures, int block, int noise_mode, const float* noise, uint32_t seed,
                         uint32_t step, const uint32_t* step_dev, void* workspace, void* peer_workspace,
                         int64_t workspace_bytes, int tile_begin, int tile_count, uint32_t* peer_flags,
                         const uint32_t* wait_flags, int wait_count, uint32_t tag, const uint32_t* epoch,
                         int32_t* x0_out, float* conf_out, mdb_stream_t stream);
/* More than 64 rows: the same call runs the tcgen05 tile GEMM over the rank's
 * columns (tile_begin even; the shard ends on a multiple of 256 columns or at
 * the end of the vocabulary; no explicit noise tensor), one record per
 * 256-column tile, mirrored into the peer's workspace.  The workspace needs
 * mdb_lmhead_tp_workspace_bytes(m, vocab) bytes; the number of flag slots a
 * shard of `cols` columns raises (the peer's wait_count) is
 * mdb_lmhead_tp_slots(m, cols). */
int64_t mdb_lmhead_tp_workspace_bytes(int m, int vocab);
int mdb_lmhead_tp_slots(int m, int cols);

/* ---- decoders with an fp32 residual: recurrent mixers, latent attention, experts ----
 *
 * Activations are MDB_BF16 or MDB_F32 (argument `dtype`); in the fp32 form every product is true fp32.  Argument
 * blocks are host structs read during the call.  A "portion" is the run of tokens a sequence brings to a step:
 * rows [cu_q[s], cu_q[s + 1]) of the step, the first of them at position start[s] of the sequence.  state_slot[s]
 * is the sequence's slot in the state pools (-1: padding entry, skipped); a sequence at position 0 starts from a
 * zero state whatever the slot holds.  Sizes with the suffix _pad are storage sizes; the surplus holds zeros. */
enum { MDB_BF16 = 0, MDB_F32 = 1 };

/* Output of a projection, columns [col, ...) of rows of `ld` elements: rows of the activation type (x), or fp32
 * split-k slices part_stride elements apart (parts) that the consumer sums and rounds. */
typedef struct {
  const void* x;
  const float* parts;
  int64_t ld, part_stride;
  int32_t nparts, col;
} mdb_rows;

enum { MDB_GEMM_PLAIN = 0, MDB_GEMM_HEADS = 1, MDB_GEMM_EXPERTS = 2 };
enum { MDB_ACT_NONE = 0, MDB_ACT_RELU2 = 1, MDB_ACT_RELU_GLU = 2, MDB_ACT_SILU = 3 };
/* y = act(x W^T).  PLAIN: x [m, k], w [n, k], y [m, n]; with RELU_GLU w is [2 n, k], gate rows first, and y =
 * relu(gate) * up (activation type, n % 128 == 0); with SILU only columns from act_from (a multiple of 4) on are
 * activated.  HEADS: head h takes columns [h k, (h + 1) k) of x, rows
 * [h n, (h + 1) n) of w and writes columns [h n, (h + 1) n) of y.  EXPERTS: rows of x and y are laid out by expert
 * in tiles of 128 (mdb_moe_plan); tile t uses rows [e n, (e + 1) n) of w, e = tile_expert[t], for t < *num_tiles;
 * m = rows of the buffers; max_rows_per_expert (0: unknown) bounds the rows in use in a tile.  y is of the
 * activation type, or fp32 with y_f32. */
typedef struct {
  int32_t dtype, form, act, y_f32;
  const void* x;
  const void* w;
  void* y;
  int64_t ldx, ldy;
  int32_t m, n, k;
  int32_t heads, experts, max_rows_per_expert;
  const int32_t* tile_expert;
  const int32_t* num_tiles;
  int32_t act_from;
} mdb_gemm_args;
int mdb_gemm(const mdb_gemm_args* args, mdb_stream_t stream);

/* residual [m][width_pad] fp32: with ids, = embed[id] * embed_scale, else *= res_scale; plus the rows of up to two
 * projections, plus sum_k moe_weight[row][k] * moe_rows[moe_slot[row][k]].  y (may be NULL) = norm(residual) * weight,
 * norm(x) = x / sqrt(mean of its first `width` columns squared + eps); weight NULL: y = residual.  With `post` the residual
 * itself becomes norm(residual) * weight, and y = residual or, with weight2, norm(residual) * weight2. */
typedef struct {
  int32_t dtype, m, width, width_pad;
  float* residual;
  const int64_t* ids;
  const void* embed;
  int64_t vocab;
  mdb_rows add[2];
  const void* moe_rows;
  int64_t moe_ld;
  const int32_t* moe_slot;
  const float* moe_weight;
  const float* weight;
  void* y;
  int64_t ldy;
  float embed_scale, eps;
  int32_t moe_top;
  int32_t post;
  const float* weight2;
  float res_scale;
} mdb_residual_norm_args;
int mdb_residual_norm(const mdb_residual_norm_args* args, mdb_stream_t stream);

/* RMSNorm of column segments of a projection into row `row` of out, or into row slots[row] (-1: skipped). */
#define MDB_MAX_RMS_SEGMENTS 4
typedef struct {
  mdb_rows src;
  const float* weight;
  void* out;
  int64_t ld_out;
  const int32_t* slots;
  int64_t num_slots;
  int32_t n, n_pad;
  float eps;
} mdb_rms_segment;
int mdb_rms_rows(int dtype, const mdb_rms_segment* segments, int nseg, int m, mdb_stream_t stream);

/* y[row][h][c] = o' / sqrt(mean over c of o'^2 + eps) * weight[h * weight_head_stride + c] * sigmoid(gate), with
 * o' = o / den[row][h] (den may be NULL: 1) */
typedef struct {
  int32_t dtype, m, heads, vdim;
  const float* o;
  const float* den;
  mdb_rows gate;
  const float* weight;
  void* y;
  int64_t ldy;
  int32_t weight_head_stride;
  float eps;
} mdb_gated_norm_args;
int mdb_gated_norm(const mdb_gated_norm_args* args, mdb_stream_t stream);

/* y[row][c] for n columns in `parts` equal parts, each normalised by its own root mean square:
 * gate_first: norm(o * silu(gate)) * weight, else norm(o) * weight * sigmoid(gate); times out_scale.  o fp32 [m][n]. */
typedef struct {
  int32_t dtype, m, n, parts, gate_first;
  float out_scale, eps;
  const float* o;
  mdb_rows gate;
  const float* weight;
  void* y;
  int64_t ldy;
} mdb_part_norm_args;
int mdb_part_norm(const mdb_part_norm_args* args, mdb_stream_t stream);

/* Key channels of a recurrent head as the state stores them (a multiple of 64; 0: not supported), and the number of
 * copies of the mLSTM maximum a head keeps. */
int mdb_scan_dim_pad(int dim);
int mdb_scan_blocks(int vdim);
/* 1 when the one-token form of mdb_scan takes this head shape */
int mdb_scan_fusable(int dim_pad, int vdim);

/* Inputs of the delta scan: causal short convolution over time per channel (weights fp32 [channels][taps], the last
 * tap is the current token's) and silu of q, k, v; q and k as unit vectors (q times dim^-1/2), beta = sigmoid(b).
 * conv_state [slot][taps - 1][channels] of the activation type, channels ordered q | k | v, holds the last inputs and is
 * moved on: in the same kernel when shift_state is set (every portion is one token), else by a
 * second one.  copy_cols columns of `copy` are written to copy_out (materialises split-k slices). */
typedef struct {
  int32_t dtype, m, bs, heads, kv_heads, dim, dim_pad, vdim, taps, channels, shift_state, copy_cols;
  mdb_rows q, k, v, b, copy;
  void* copy_out;
  int64_t copy_ld;
  const float* conv_q;
  const float* conv_k;
  const float* conv_v;
  void* conv_state;
  int64_t conv_slot_stride, num_slots;
  const int32_t* row_seq;
  const int32_t* cu_q;
  const int32_t* start;
  const int32_t* state_slot;
  float* q_out;    /* [m][kv_heads][dim_pad] */
  float* k_out;
  float* v_out;    /* [m][heads][vdim] */
  float* beta_out; /* [m][heads] */
} mdb_delta_prep_args;
int mdb_delta_prep(const mdb_delta_prep_args* args, mdb_stream_t stream);

/* g [m][heads][dim_pad] = exp(-exp(a_log[h]) * softplus(x + dt_bias)), x [m] rows of heads * dim columns; scalars
 * [m][heads][4] = (k . q, (g k_prev) . k, (g k_prev) . q, beta) with the outputs of mdb_delta_prep; the products with the
 * token before are written for the odd tokens of every portion. */
typedef struct {
  int32_t m, heads, kv_heads, dim, dim_pad;
  const float* x;
  int64_t ldx;
  const float* a_log;
  const float* dt_bias;
  const float* q;
  const float* k;
  const float* beta;
  float* g;
  float* scalars;
  const int32_t* row_seq;
  const int32_t* cu_q;
} mdb_decay_args;
int mdb_channel_decay(const mdb_decay_args* args, mdb_stream_t stream);

/* Inputs of the mLSTM scan: q times dim^-1/2, k, v as fp32 rows; log_i = cap tanh((i + bias_i) / cap), log_f =
 * logsigmoid(cap tanh((f + bias_f) / cap)). */
typedef struct {
  int32_t dtype, m, heads, dim, dim_pad, vdim;
  mdb_rows q, k, v, i, f;
  const float* bias_i;
  const float* bias_f;
  float* q_out;
  float* k_out;
  float* v_out;
  float* log_i; /* [m][heads] */
  float* log_f;
  float cap;
} mdb_mlstm_prep_args;
int mdb_mlstm_prep(const mdb_mlstm_prep_args* args, mdb_stream_t stream);

/* Inputs of the decay scan (a linear recurrence with one decay per head): v [m][heads][vdim], k, q [m][kv_heads][dim_pad]
 * = silu of the projections or, with taps > 0, silu of a causal short convolution with bias over time (channels ordered
 * v | k | q; conv fp32 [channels][taps], the last tap is the current token's; conv_state as in mdb_delta_prep).  With dt:
 * step = softplus(dt + dt_bias), decay = exp(-exp(a_log) * step); else step = 1, decay = decay_const[h].  for_chunks: q, k, v
 * leave in bf16 and decay_out holds the logarithm, as mdb_chunk_scan takes them. */
typedef struct {
  int32_t dtype, m, bs, heads, kv_heads, dim, dim_pad, vdim, taps, channels, shift_state, for_chunks;
  mdb_rows q, k, v, dt;
  const float* conv;
  const float* conv_bias;
  void* conv_state;
  int64_t conv_slot_stride, num_slots;
  const int32_t* row_seq;
  const int32_t* cu_q;
  const int32_t* start;
  const int32_t* state_slot;
  const float* a_log;
  const float* dt_bias;
  const float* decay_const;
  void* q_out; /* fp32, or bf16 with for_chunks */
  void* k_out;
  void* v_out;
  float* decay_out; /* [m][heads] */
  float* step_out;
} mdb_decay_prep_args;
int mdb_decay_prep(const mdb_decay_prep_args* args, mdb_stream_t stream);

/* The recurrences over every sequence's portion; state [slot][heads][vdim][dim_pad] fp32 is read and written.
 * DELTA: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q; beta comes
 * with the scalars of mdb_channel_decay, in the fused form as s0.  MLSTM: m' = max(f + m, i);
 * S, n <- exp(f + m - m') (.) + exp(i - m') k (v^T, 1); o = S^T q, den [m][heads] = max(|n . q|, exp(-m')) + 1e-6;
 * s0 = i, s1 = f; its state has one more column per head (vdim + 1), which is n; mstate [slot][heads][mdb_scan_blocks].
 * DECAY: S <- s0 S + s1 k v^T; o = S^T q + skip[h] v (skip may be NULL); with `fused` only the form changes, out is written.
 * out [m][heads][vdim] fp32; with `fused` (every portion is one token) the decay comes from raw_decay + dt_bias and
 * a_log, and y = the gated norm of o / den (as mdb_gated_norm) is written instead. */
enum { MDB_SCAN_DELTA = 0, MDB_SCAN_MLSTM = 1, MDB_SCAN_DECAY = 2 };
typedef struct {
  int32_t mode, dtype, fused, bs, heads, kv_heads, dim, dim_pad, vdim;
  float eps;
  const float* q;
  const float* k;
  const float* v;
  const float* g;
  const float* s0;
  const float* s1;
  float* state;
  int64_t state_slot_stride, num_slots;
  float* mstate;
  const float* scalars; /* DELTA: of mdb_channel_decay */
  float* den;         /* MLSTM */
  const int32_t* cu_q;
  const int32_t* start;
  const int32_t* state_slot;
  float* out;
  mdb_rows raw_decay; /* fp32 */
  const float* a_log;
  const float* dt_bias;
  mdb_rows gate;
  const float* norm;
  int64_t norm_head_stride;
  void* y;
  int64_t ldy;
  const float* skip; /* DECAY */
} mdb_scan_args;
int mdb_scan(const mdb_scan_args* args, mdb_stream_t stream);

/* The decay scan over prompt portions in chunks of 64 tokens on the tensor cores: bf16 rows of ldq / ldk elements with head
 * g of q and k at column g * dim (dim a multiple of 8, missing channels up to dim_pad count as zeros) and rows of ldv elements
 * with head h of v at column h * vdim; log_decay (at least -104) and step are rows of heads, ld_scalars elements apart
 * (0: the same for every token); state and out as in mdb_scan; max_q = longest portion, m = rows.  Key heads of exactly 64 or
 * 128 channels take chunks of 128 tokens where a portion is longer than 64. */
typedef struct {
  int32_t m, bs, heads, kv_heads, dim, dim_pad, vdim, max_q;
  const void* q;
  const void* k;
  const void* v;
  int64_t ldq, ldk, ldv, ld_scalars;
  const float* log_decay;
  const float* step;
  const float* skip; /* [heads], may be NULL */
  float* state;
  int64_t state_slot_stride, num_slots;
  const int32_t* cu_q;
  const int32_t* start;
  const int32_t* state_slot;
  float* out;
} mdb_chunk_scan_args;
/* 1 when mdb_chunk_scan takes this head shape */
int mdb_chunk_scan_supported(int dim_pad, int vdim);
int mdb_chunk_scan(const mdb_chunk_scan_args* args, mdb_stream_t stream);

/* Group-limited top-k routing of fp32 logits [m][experts]: ids and weights [m][top]; rows with row_slot < 0 (may be
 * NULL) get ids -1. */
typedef struct {
  int32_t m, experts, top, groups, keep;
  mdb_rows logits; /* fp32 */
  const int32_t* row_slot;
  int32_t* ids;
  float* weights;
} mdb_moe_route_args;
int mdb_moe_route(const mdb_moe_route_args* args, mdb_stream_t stream);

/* Lays the (token, k) pairs out by expert in tiles of 128 rows: slot [m][top] (row of the pair, -1: none), row_token
 * [max_tiles * 128] (-1: padding), tile_expert [max_tiles], num_tiles [1]. */
typedef struct {
  int32_t m, top, experts, max_tiles;
  const int32_t* ids;
  int32_t* slot;
  int32_t* row_token;
  int32_t* tile_expert;
  int32_t* num_tiles;
} mdb_moe_plan_args;
int mdb_moe_plan(const mdb_moe_plan_args* args, mdb_stream_t stream);
/* Most tiles m rows with `top` experts each can need. */
int mdb_moe_max_tiles(int m, int top, int experts);
int mdb_moe_gather(int dtype, const void* x, int64_t ldx, void* out, int width, const int32_t* row_token,
                   const int32_t* num_tiles, int max_tiles, mdb_stream_t stream);

/* Causal attention over cached latents (cache [pages * 256][width], one row per token, key and value of every head
 * alike): q, out [m][heads][width]; the row at position p of its sequence sees keys 0 .. p. */
int64_t mdb_latent_attn_workspace_bytes(int m, int heads, int width, int nsplit);
int mdb_latent_attn(int dtype, const void* q, const void* cache, void* out, const int32_t* block_table, int table_stride,
                    const int32_t* row_seq, const int32_t* row_pos, int m, int heads, int width, int num_pages, float scale,
                    int nsplit, void* workspace, int64_t workspace_bytes, mdb_stream_t stream);
/* out [total][width] = the latents of positions 0 .. cu[s + 1] - cu[s] - 1 of every sequence, in order. */
int mdb_gather_latents(int dtype, const void* cache, const int32_t* block_table, int table_stride, int num_pages,
                       const int32_t* cu, int nseq, int total, void* out, int width, mdb_stream_t stream);
/* Causal attention over packed rows (bf16, head size 128): the queries of sequence s are its last cu_q[s + 1] -
 * cu_q[s] tokens, the keys all of them (cu_k). */
int mdb_attn_causal_varlen(const void* q, int64_t q_stride, const void* k, int64_t k_stride, const void* v, int64_t v_stride,
                           void* out, int64_t out_stride, const int32_t* cu_q, const int32_t* cu_k, int nseq, int max_q,
                           int64_t total_q, int64_t total_k, int hq, int hkv, float scale, mdb_stream_t stream);

/* Queries and keys of rotary attention: per head RMSNorm (weight fp32 [dim]) and rotation of channel pairs (2 i, 2 i + 1),
 * i < rot_dims / 2, by row_pos * inv_freq[i].  q_out [m][heads][dim_pad]; k and the values v as they come go to row
 * slots[row] (-1: skipped) of the caches [slots][kv_heads][dim_pad]. */
typedef struct {
  int32_t dtype, m, heads, kv_heads, dim, dim_pad, rot_dims;
  float eps;
  mdb_rows q, k, v;
  const float* q_norm;
  const float* k_norm;
  const double* inv_freq;
  const int32_t* row_pos;
  const int32_t* slots;
  int64_t num_slots;
  void* q_out;
  void* k_cache;
  void* v_cache;
} mdb_rotary_commit_args;
int mdb_rotary_commit(const mdb_rotary_commit_args* args, mdb_stream_t stream);

/* Causal grouped-query attention over the paged caches of mdb_rotary_commit: the row at position p of its sequence sees
 * keys max(0, p - window + 1) .. p (window 0: all).  sink: one more term exp(0) in the softmax's denominator.  Head h's
 * output is multiplied by out_scale and, with a gate, by sigmoid(gate[row][h]); out [m] rows of ld_out elements, head h at
 * column h * dim.  max_q = longest portion, max_ctx = longest context of the step (bounds); portions of many tokens take
 * the tensor-memory kernel (bf16, dim_pad 128), which needs cu_q and start. */
typedef struct {
  int32_t dtype, m, bs, heads, kv_heads, dim, dim_pad, window, sink, max_q, nsplit;
  float scale, out_scale;
  const void* q;
  const void* k_cache;
  const void* v_cache;
  const int32_t* block_table;
  const int32_t* row_seq;
  const int32_t* row_pos;
  const int32_t* cu_q;
  const int32_t* start;
  int32_t table_stride, num_pages;
  mdb_rows gate;
  void* out;
  int64_t ld_out;
  void* workspace;
  int64_t workspace_bytes;
} mdb_window_attn_args;
int64_t mdb_window_attn_workspace_bytes(int m, int heads, int dim_pad, int nsplit);
int mdb_window_attn(const mdb_window_attn_args* args, mdb_stream_t stream);

/* token = argmax of logits / temperature + Gumbel noise (seed, *step_dev, row), or of the logits where the row's
 * temperature is 0; status_out (may be NULL) receives and clears the device status word. */
int mdb_pick_token(const float* logits, int64_t ld, int m, int vocab, const float* temperatures, uint32_t seed,
                   const uint32_t* step_dev, int64_t* out, uint32_t* status_out, mdb_stream_t stream);

#ifdef __cplusplus
}
#endif
#endif /* MDB200_H */
