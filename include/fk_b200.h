/*
 * fk_b200.h -- C ABI of libfk_b200.so: the decode hot path of the FastKernels
 * nano-vllm-style serving engine as hand-written sm_100a CUDA kernels.
 *
 * Conventions (all entry points):
 *   - plain pointers and sizes only; every pointer is a DEVICE pointer unless
 *     its comment says "host";
 *   - strides are in ELEMENTS of the tensor's dtype, sizes in elements unless
 *     the name ends in _bytes;
 *   - the activation / cache dtype is bf16 (2 bytes); accumulation is fp32;
 *   - `stream` is a cudaStream_t (CUstream) passed as an opaque pointer; the
 *     call only enqueues work on it: no allocation, no host synchronisation,
 *     so every call can be captured into a CUDA graph;
 *   - the return value is FK_OK (0) or a negative fk_status code after
 *     host-side argument validation; nothing throws.  fk_last_error() gives
 *     the message of the last failing call on the calling thread;
 *   - kernels never trap: device-side problems (an out-of-range slot or page
 *     id, a wait that ran out) are recorded in the optional `status` word
 *     (one int32 in device memory, 0 = clean) and the offending access is
 *     skipped.
 *
 * Each declaration cites the reference interface it replaces
 * (paths relative to the reference repository root).
 */
#ifndef FK_B200_H_
#define FK_B200_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef void* fk_stream_t; /* cudaStream_t */

enum fk_status {
  FK_OK = 0,
  FK_ERR_INVALID_ARG = -1, /* null pointer, negative size, bad stride        */
  FK_ERR_UNSUPPORTED = -2, /* a shape this build has no kernel for            */
  FK_ERR_WORKSPACE = -3,   /* workspace pointer null or too small             */
  FK_ERR_ALIGNMENT = -4,   /* pointer / stride breaks a 16-byte requirement   */
  FK_ERR_CUDA = -5         /* a CUDA runtime / driver call failed             */
};

/* Device-side status bits written (atomicOr) into the optional status word. */
enum fk_device_status {
  FK_DEV_BAD_SLOT = 1,     /* slot_mapping entry >= num_slots: row skipped    */
  FK_DEV_BAD_PAGE = 2,     /* block_table entry outside [0, num_blocks)       */
  FK_DEV_WAIT_TIMEOUT = 4, /* a bounded mbarrier / flag wait ran out          */
  FK_DEV_BAD_POSITION = 8, /* position outside [0, max_position)              */
  FK_DEV_TMEM_BASE = 16    /* tensor memory was not handed out from column 0  */
};

/* Activation of a gated feed-forward, act(gate) * up. */
enum fk_activation {
  FK_ACT_SILU = 0,
  FK_ACT_GELU_TANH = 1     /* 0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))) */
};

/* Library version: major*10000 + minor*100 + patch. */
int fk_version(void);

/* Message of the last failing call on this thread ("" if none). Host pointer,
 * valid until the next failing call on the same thread. */
const char* fk_last_error(void);

/* Programmatic dependent launch between the library's kernels (default on; the
 * environment variable FK_B200_PDL=0 turns it off).  Returns the previous
 * setting.  With it on, a kernel's launch latency and prologue overlap the tail
 * of the kernel before it on the same stream; results are identical. */
int fk_set_pdl(int enabled);

/* Number of kernels this library has launched since load (host counter). */
int64_t fk_launch_count(void);

/* ------------------------------------------------------------------------
 * KV-cache store.
 * Replaces StoreKVCache.forward(key, value, k_cache, v_cache, slot_mapping)
 * (fastkernels/tasks/baseline/L1/store_kvcache.py:71-82, kernel 16-35):
 *   for every token i with slot = slot_mapping[i] >= 0:
 *     k_cache.view(-1, row_elems)[slot] = key[i]; same for value.
 * key/value: [num_tokens, row_elems] with row strides key_stride/value_stride
 * (views into a packed qkv buffer are fine); caches: contiguous
 * [num_slots, row_elems].  slot_mapping is int32 (slot_is_int64 == 0) or
 * int64.  Rows with slot < 0 are skipped; rows with slot >= num_slots are
 * skipped and flagged FK_DEV_BAD_SLOT.  Raw 16-bit copy: bit-exact.
 * ---------------------------------------------------------------------- */
int fk_store_kvcache(const void* key, const void* value, void* k_cache,
                     void* v_cache, const void* slot_mapping,
                     int slot_is_int64, int64_t num_tokens, int64_t row_elems,
                     int64_t key_stride, int64_t value_stride,
                     int64_t num_slots, int32_t* status, fk_stream_t stream);

/* HND pool [num_blocks, num_kv_heads, page_size, head_dim].  Replaces
 * StoreKVCacheHND.forward (fastkernels/tasks/baseline/L1/store_kvcache.py:85-101,
 * kernel 38-68): slot -> block = slot / page_size, offset = slot % page_size.
 * key/value: [num_tokens, num_kv_heads, head_dim], heads dense, token strides
 * given.  Same skipping / flagging rules as fk_store_kvcache.  Bit-exact. */
int fk_store_kvcache_hnd(const void* key, const void* value, void* k_cache,
                         void* v_cache, const void* slot_mapping,
                         int slot_is_int64, int64_t num_tokens, int num_kv_heads,
                         int head_dim, int64_t key_stride, int64_t value_stride,
                         int page_size, int64_t num_blocks, int32_t* status,
                         fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Paged GQA decode attention (one query token per sequence).
 * Replaces FlashAttnDecode.forward(q, k_cache, v_cache, cache_seqlens,
 *   block_table=..., softmax_scale=..., causal=True, max_seq_len=...)
 * (fastkernels/tasks/baseline/L1/flash_attn_decode.py:113-181); same maths as
 * Attention._decode_torch (fastkernels/tasks/baseline/L2/attention_impl.py:
 * 598-664): out[i,h] = softmax(scale * q[i,h] . K_i[:L_i, h/g]^T) V_i[:L_i, h/g]
 * with K_i/V_i gathered through block_tables[i, p]*block_size + offset.
 *
 * q:   [batch, num_q_heads, head_dim], token stride q_stride_token, heads
 *      contiguous (stride head_dim).  out likewise with out_stride_token.
 * k_cache/v_cache: paged pool, contiguous within a block, blocks
 *      kv_block_stride elements apart; kv_layout 0 = NHD
 *      [num_blocks, block_size, num_kv_heads, head_dim] (the flash-attn path),
 *      kv_layout 1 = HND [num_blocks, num_kv_heads, block_size, head_dim] (what
 *      TRTLLMDecode reads, fastkernels/tasks/baseline/L1/flashinfer_decode.py:
 *      44-107, the reference's default on B200 with page size 16).
 * context_lens: [batch] int32 (0 = padded row: output row is zero-filled).
 * block_tables: [batch, >= ceil(L/block_size)] int32, rows
 *      block_table_stride apart (may exceed the live column count).
 * max_splits: upper bound on KV splits per sequence the workspace was sized
 *      for (fk_paged_decode_attn_workspace_bytes).  The split size is chosen
 *      on the device from context_lens, so one captured launch serves every
 *      replay.
 * Supported: head_dim 128, block_size 16, 32 or a multiple of 64,
 * num_q_heads/num_kv_heads in {1,2,4,8,16}, bf16.
 * Launches: plan + main + merge kernel; a small call (batch * num_kv_heads <= SM
 *      count and block tables of at most 2048 tokens) is a single launch in which
 *      every (sequence, KV head) pair has its own CTA and nothing is split.
 * ---------------------------------------------------------------------- */
size_t fk_paged_decode_attn_workspace_bytes(int batch, int num_q_heads,
                                            int head_dim, int max_splits);

int fk_paged_decode_attn(const void* q, int64_t q_stride_token, void* out,
                         int64_t out_stride_token, const void* k_cache,
                         const void* v_cache, int64_t num_blocks,
                         int block_size, int64_t kv_block_stride, int kv_layout,
                         const int32_t* context_lens,
                         const int32_t* block_tables,
                         int64_t block_table_stride, int batch,
                         int num_q_heads, int num_kv_heads, int head_dim,
                         float softmax_scale, int max_splits, void* workspace,
                         size_t workspace_bytes, int32_t* status,
                         fk_stream_t stream);

/* The split schedule depends only on context_lens, which every layer of a decode
 * step shares (the engine sets one Context per step,
 * fastkernels/infra/engine.py:6057-6063).  fk_paged_decode_attn_plan computes it
 * once into the workspace; fk_paged_decode_attn_planned is fk_paged_decode_attn
 * without the plan launch and may be called for any number of layers afterwards
 * with the same workspace, context_lens, block_tables, batch, head counts and
 * max_splits (each call leaves the schedule ready for the next). */
int fk_paged_decode_attn_plan(const int32_t* context_lens,
                              const int32_t* block_tables,
                              int64_t block_table_stride, int block_size, int batch,
                              int num_q_heads, int num_kv_heads, int head_dim,
                              int max_splits, void* workspace,
                              size_t workspace_bytes, int32_t* status,
                              fk_stream_t stream);

int fk_paged_decode_attn_planned(const void* q, int64_t q_stride_token, void* out,
                                 int64_t out_stride_token, const void* k_cache,
                                 const void* v_cache, int64_t num_blocks,
                                 int block_size, int64_t kv_block_stride,
                                 int kv_layout,
                                 const int32_t* context_lens,
                                 const int32_t* block_tables,
                                 int64_t block_table_stride, int batch,
                                 int num_q_heads, int num_kv_heads, int head_dim,
                                 float softmax_scale, int max_splits,
                                 void* workspace, size_t workspace_bytes,
                                 int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * RMSNorm and fused residual-add + RMSNorm.
 * Replace RMSNorm.forward(x, residual=None)
 * (fastkernels/tasks/baseline/L1/rms_norm.py:153-164; kernels
 * fastkernels/tasks/baseline/L1/rms_norm.cu:1251-1336 and 1342-1410):
 *   fk_rmsnorm:  out = bf16(float(x) * rsqrt(mean(x^2)+eps) * float(w))
 *     rows of `cols` elements; x rows x_stride apart (per-head q/k norm on a
 *     strided [N, H, D] view passes rows = N*H with the 3-D form below);
 *   fk_fused_add_rmsnorm (in place, both tensors):
 *     residual = bf16(x + residual); x = bf16(float(residual) * rsqrt(...) * w)
 * ---------------------------------------------------------------------- */
int fk_rmsnorm(const void* x, int64_t x_stride_outer, int64_t x_stride_inner,
               int64_t inner, void* out, int64_t out_stride_outer,
               int64_t out_stride_inner, const void* weight, float eps,
               int64_t outer, int64_t cols, fk_stream_t stream);

int fk_fused_add_rmsnorm(void* x, int64_t x_stride, void* residual,
                         int64_t residual_stride, const void* weight,
                         float eps, int64_t rows, int64_t cols,
                         fk_stream_t stream);

/* ------------------------------------------------------------------------
 * NeoX rotary embedding, in place on query and key.
 * Replaces RotaryEmbedding.forward(positions, query, key)
 * (fastkernels/tasks/baseline/L1/rotary_emb.py:179-191; kernel
 * fastkernels/tasks/baseline/L1/rotary_emb.cu:332-423):
 *   (x_i, x_{i+D/2}) <- (x_i c - x_{i+D/2} s, x_{i+D/2} c + x_i s),
 *   c,s = cache[pos, i], cache[pos, D/2+i] rounded to bf16, fp32 maths, one
 *   rounding.  cos_sin_cache: [max_position, head_dim], fp32
 *   (cache_is_fp32 = 1; rounded to bf16 in the kernel, as the reference's
 *   per-call cast does) or bf16.  positions: [num_tokens] int64.
 * ---------------------------------------------------------------------- */
int fk_rope_neox(const int64_t* positions, void* query, int64_t q_stride,
                 int num_q_heads, void* key, int64_t k_stride,
                 int num_kv_heads, int head_dim, const void* cos_sin_cache,
                 int cache_is_fp32, int64_t max_position, int64_t num_tokens,
                 int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Fused QKV split + optional per-head q/k RMSNorm + NeoX RoPE + KV store.
 * Replaces, in one pass over the packed projection output, the chain in
 * LlamaAttention.forward (fastkernels/tasks/baseline/L2/attention.py:113-156):
 *   qkv.split -> [q_norm/k_norm] -> rotary_emb -> Attention.forward_impl's
 *   StoreKVCache (fastkernels/tasks/baseline/L2/attention_impl.py:313-325).
 * qkv: [num_tokens, (Hq + 2 Hkv) * D] with row stride qkv_stride; q and k are
 * rotated IN PLACE inside qkv (so a later reader of the q view sees the same
 * values the reference produces); rotated k and raw v are also written to
 * k_cache/v_cache at slot_mapping[i] (int32; < 0 skips the store).
 * kv_layout 0 = NHD cache (block_size unused), 1 = HND cache with pages of
 * block_size tokens.
 * q_norm_weight / k_norm_weight: [D] bf16 or NULL (no per-head norm).
 * Rounding points match the unfused chain: normed value rounded to bf16, then
 * rotated in fp32 and rounded once.
 * ---------------------------------------------------------------------- */
int fk_qkv_rope_store(void* qkv, int64_t qkv_stride, int num_q_heads,
                      int num_kv_heads, int head_dim,
                      const int64_t* positions, const void* cos_sin_cache,
                      int cache_is_fp32, int64_t max_position,
                      const void* q_norm_weight, const void* k_norm_weight,
                      float norm_eps, void* k_cache, void* v_cache,
                      const int32_t* slot_mapping, int64_t num_slots,
                      int block_size, int kv_layout, int64_t num_tokens,
                      int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * SiLU-and-multiply.  Replaces SiluAndMul.forward(x)
 * (fastkernels/tasks/baseline/L1/silu_and_mul.py:32-35; kernel
 * fastkernels/tasks/baseline/L1/silu_and_mul.cu:715-740):
 *   out[t, j] = bf16(float(bf16(silu(x[t, j]))) * float(x[t, d + j]))
 * x: [rows, 2*d] row stride x_stride; out: [rows, d] row stride out_stride.
 * ---------------------------------------------------------------------- */
int fk_silu_and_mul(const void* x, int64_t x_stride, void* out,
                    int64_t out_stride, int64_t rows, int64_t d,
                    fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Dense projection y = x W^T (+ bias): bf16 x bf16 -> fp32 (TMEM) -> bf16.
 * Replaces Matmul.forward(input, weight, bias)
 * (fastkernels/tasks/baseline/L1/linear.py:13-17) and the F.linear calls of
 * {QKV,MergedColumn,Column,Row}ParallelLinear.forward
 * (fastkernels/tasks/baseline/L2/parallel_linear.py:78-81,157-160,237-240,
 * 327-335).  x: [m, k] row stride x_stride; w: [n, k] row-major contiguous
 * (the nn.Linear layout); y: [m, n] row stride y_stride; bias [n] or NULL.
 * k % 64 == 0, n % 8 == 0.  m <= 256 (decode) runs the weight-streaming kernel;
 * m > 256 (prefill) runs a 256 x 256 tile kernel, needs no workspace
 * (fk_gemm_bf16_workspace_bytes returns 0) and 16-byte aligned rows of y.
 * workspace: fk_gemm_bf16_workspace_bytes(m, n, k) bytes, 256-byte aligned,
 * ZERO-INITIALISED once by the caller (cudaMemset) before its first use: it holds
 * the stream-K flags and fp32 partial tiles, and every call leaves it zeroed
 * again, so one buffer can serve all GEMMs issued on one stream.  Two calls that
 * may run concurrently need separate workspaces.
 * After FK_DEV_WAIT_TIMEOUT was reported in `status` the results of that call are
 * undefined and a late contributor may have left a flag raised: zero the first
 * 1024 bytes of the workspace again (stream-ordered) before the next call.
 * ---------------------------------------------------------------------- */
size_t fk_gemm_bf16_workspace_bytes(int64_t m, int64_t n, int64_t k);

int fk_gemm_bf16(const void* x, int64_t x_stride, const void* w,
                 const void* bias, void* y, int64_t y_stride, int64_t m,
                 int64_t n, int64_t k, void* workspace,
                 size_t workspace_bytes, int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Gate/up projection fused with SiLU-and-multiply: y = silu(x Wg^T) * (x Wu^T)
 * with W = [Wg; Wu] the merged [n, k] matrix (n/2 gate rows, then n/2 up rows).
 * Replaces the pair MergedColumnParallelLinear.forward
 *   (fastkernels/tasks/baseline/L2/parallel_linear.py:157-160) + SiluAndMul.forward
 *   (fastkernels/tasks/baseline/L1/silu_and_mul.py:32-35) as LlamaMLP.forward
 *   chains them (fastkernels/tasks/baseline/L2/llama_mlp.py:35-38).
 * Rounding points are those of the two separate ops: both projection outputs are
 * rounded to bf16 (+ bias, [n] or null), silu(gate) is rounded to bf16, the
 * product once more.  y is [m, n/2] bf16; the [m, n] intermediate never exists.
 * Same workspace as fk_gemm_bf16(m, n, k).  Only shapes that take the persistent
 * stream-K schedule have this single-launch form (m <= 256, n % 128 == 0, more
 * weight tiles than half the SMs): fk_gemm_bf16_silu_mul_fusable says which;
 * other shapes return FK_ERR_UNSUPPORTED and the caller runs the two ops.
 * ---------------------------------------------------------------------- */
int fk_gemm_bf16_silu_mul_fusable(int64_t m, int64_t n, int64_t k);
int fk_gemm_bf16_silu_mul(const void* x, int64_t x_stride, const void* w,
                          const void* bias, void* y, int64_t y_stride, int64_t m,
                          int64_t n, int64_t k, void* workspace,
                          size_t workspace_bytes, int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Persistent decode block: the kernels a decoder layer runs between two
 * attention calls, as ONE launch (one persistent CTA per SM) that walks a
 * program of up to 8 phases.  It computes what the reference computes with
 *   RowParallelLinear.forward (o_proj)     fastkernels/tasks/baseline/L2/parallel_linear.py:327-335
 *   RMSNorm.forward(x, residual)            fastkernels/tasks/baseline/L1/rms_norm.py:153-164
 *   LlamaMLP.forward                        fastkernels/tasks/baseline/L2/llama_mlp.py:35-38
 *   LlamaDecoderLayer.forward (norm order)  fastkernels/tasks/baseline/L3/llama_decoder.py:34-42
 *   LlamaAttention.forward up to the attention call (qkv_proj, q/k norm, RoPE)
 *                                           fastkernels/tasks/baseline/L2/attention.py:113-150
 *   StoreKVCache.forward                    fastkernels/tasks/baseline/L1/store_kvcache.py:71-82
 * with the rounding points of the separate entry points above (fk_gemm_bf16,
 * fk_gemm_bf16_silu_mul, fk_fused_add_rmsnorm / fk_rmsnorm, fk_qkv_rope_store).
 * Phases run in order; each sees everything the earlier ones wrote (a grid-wide
 * barrier with bounded waits -> FK_DEV_WAIT_TIMEOUT), while the weight tiles of
 * later projections are already being fetched.  Phase kinds and the fields read:
 *   FK_PHASE_GEMM            y[m, n] = x[m, k] w[n, k]^T (+ bias[n])
 *   FK_PHASE_GEMM_SILU_MUL   y[m, n/2] = silu(x wg^T) * (x wu^T), w = [wg; wu], n % 128 == 0
 *       x, x_stride, w, bias, y, y_stride, n, k              (k % 64 == 0)
 *   FK_PHASE_ADD_RMSNORM     residual = bf16(x + residual) (x null: nothing added);
 *                            y = rmsnorm(residual) * norm_weight over n columns
 *       x, x_stride, residual, residual_stride, norm_weight, eps, y, y_stride, n
 *   FK_PHASE_QKV_ROPE_STORE  fk_qkv_rope_store on x = packed qkv rows (head_dim 128,
 *                            bf16 cos/sin cache), at most once per launch
 *       x, x_stride, num_q_heads, num_kv_heads, head_dim, positions, cos_sin_cache,
 *       cache_is_fp32 (must be 0), max_position, q_norm_weight, k_norm_weight, eps,
 *       k_cache, v_cache, slot_mapping, num_slots, block_size, kv_layout
 * m <= 128 rows, at most 4 projections per launch.  workspace: fk_decode_block_
 * workspace_bytes(m) bytes, 256-byte aligned, zero-initialised once; a launch
 * leaves it zeroed (unless a wait timed out: re-zero it then).  Launches that
 * share a workspace must not overlap on the GPU.  Every CTA must be resident for
 * the barriers to complete: the grid is one CTA per SM, so give the kernel the
 * whole device (no other long-running kernel alongside).
 * ---------------------------------------------------------------------- */
enum fk_block_phase_kind {
  FK_PHASE_GEMM = 1,
  FK_PHASE_GEMM_SILU_MUL = 2,
  FK_PHASE_ADD_RMSNORM = 3,
  FK_PHASE_QKV_ROPE_STORE = 4
};
typedef struct fk_block_phase {
  int32_t kind;
  const void* x; int64_t x_stride;
  const void* w; const void* bias;
  void* y; int64_t y_stride;
  int64_t n, k;
  void* residual; int64_t residual_stride;
  const void* norm_weight; float eps;
  int32_t num_q_heads, num_kv_heads, head_dim;
  const int64_t* positions;
  const void* cos_sin_cache; int32_t cache_is_fp32; int64_t max_position;
  const void* q_norm_weight; const void* k_norm_weight;
  void* k_cache; void* v_cache;
  const int32_t* slot_mapping; int64_t num_slots;
  int32_t block_size, kv_layout;
} fk_block_phase;
size_t fk_decode_block_workspace_bytes(int64_t m);
int fk_decode_block(const fk_block_phase* phases, int num_phases, int64_t m,
                    void* workspace, size_t workspace_bytes, int32_t* status,
                    fk_stream_t stream);

/* ------------------------------------------------------------------------
 * fk_gemm_bf16 for callers that cannot allocate device memory.
 * No counterpart in the reference: this entry point exists for hosts that get
 * their tensors from someone else and may not call cudaMalloc themselves -- a
 * plugin running inside another runtime's memory pool, code on a stream that is
 * being captured, a sandbox whose allocator is off limits.  Same arguments and
 * results as fk_gemm_bf16 minus the workspace: the stream-K scratch is a
 * ~5 MiB array built into the library image (each GPU that loads the library
 * keeps it until the process exits).
 *   - limit: m <= 64 (the scratch is sized for it); a larger m returns
 *     FK_ERR_UNSUPPORTED and says so in fk_last_error();
 *   - the call itself allocates nothing: no cudaMalloc / cudaFree, no allocating
 *     library routine;
 *   - the FIRST call on each device looks up the array's device address
 *     (cudaGetSymbolAddress); the device the stream belongs to must be the
 *     current device.  Make that first call before any stream capture begins: a
 *     first call on a stream that is being captured returns FK_ERR_UNSUPPORTED.
 *     The flag words need no clearing at set-up: the array is zero when the
 *     library is loaded;
 *   - every call shares the one array, which keeps the previous call's partial
 *     tiles (only the flag words need to be zero, and each call leaves them
 *     zero): calls that overlap on the GPU -- two streams, two host threads --
 *     race on it; issue them on one stream, or use fk_gemm_bf16 with separate
 *     workspaces.
 * ---------------------------------------------------------------------- */
int fk_gemm_bf16_static(const void* x, int64_t x_stride, const void* w,
                        const void* bias, void* y, int64_t y_stride, int64_t m,
                        int64_t n, int64_t k, int32_t* status,
                        fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Greedy sampling over the lm-head logits: per row the maximum (as fp32) and
 * its index.  Replaces lm_logits[:bs].max(dim=-1) in the captured decode graph
 * (fastkernels/infra/engine.py:6994-6996).  Ties go to the LOWEST index; NaN
 * never wins.  x: [rows, cols] bf16 row stride x_stride; out_val [rows] fp32
 * (may be NULL); out_idx [rows] int64.
 * ---------------------------------------------------------------------- */
int fk_argmax_bf16(const void* x, int64_t x_stride, int64_t rows, int64_t cols,
                   float* out_val, int64_t* out_idx, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Tensor-parallel all-reduce fused with residual add + RMSNorm, over peer memory.
 * Replaces AllReduce.forward (fastkernels/tasks/baseline/L1/allreduce.py:37-55,
 * one-shot kernel fastkernels/tasks/baseline/L1/allreduce.cu:193-212) followed by
 * RMSNorm.forward(x, residual) (fastkernels/tasks/baseline/L1/rms_norm.py:153-164);
 * the reference's own fused form is
 * fastkernels/tasks/baseline/L2/flashinfer_allreduce_fusion.py:227-297.
 *
 * Communication buffer (one per rank, same size on all ranks):
 *   fk_comm_alloc        cudaMalloc + zero; layout = fk_comm_header_bytes() of flag
 *                        words, then caller-defined data slots
 *   fk_comm_ipc_export   64-byte CUDA IPC handle of the buffer (send to the peers)
 *   fk_comm_ipc_import   map a peer's buffer, returns its local address
 * These four are set-up calls (they allocate / map; not for use during capture).
 *
 * fk_allreduce_add_rmsnorm: bases = HOST array of nranks device addresses, entry r
 * being rank r's buffer as mapped in this process (bases[rank] is the local one).
 * Each rank's partial [rows, cols] bf16 (rows dense) sits at bases[r] +
 * slot_offset_bytes.  Computes, identically on every rank,
 *   s = bf16(sum_r y_r) (fp32, rank order); residual = bf16(s + residual) in place;
 *   out = bf16(float(residual) * rsqrt(mean(residual^2) + eps) * float(weight)).
 * Callers alternate between (at least) two slots on consecutive calls; all ranks
 * must issue the same sequence of calls.  rows <= 512, cols % 8 == 0, <= 16384.
 * Waits on peers are bounded (2 s) and reported as FK_DEV_WAIT_TIMEOUT.
 *
 * fk_allreduce_add_rmsnorm_staged: the same result (bit for bit) through a
 * two-stage exchange, for payloads where pulling every rank's rows costs more
 * than a second flag round -- the regime in which the reference switches from its
 * one-stage to its two-stage kernel
 * (fastkernels/tasks/baseline/L1/allreduce.cu:214-250, switch-over 404-415).
 * fk_allreduce_two_stage_preferred is this build's own switch-over, set from
 * measurements on B200: one stage at every decode payload, two from 4 MiB on 8 ranks.  Row i is reduced by rank
 * i % nranks alone, which pushes the bf16 sum into rows*cols*2 bytes of staging at
 * bases[r] + staging_offset_bytes of every peer r; the staging rows must not
 * overlap the data slot, and calls alternate between two staging areas exactly as
 * they alternate between two slots.  Calls of both kinds may be mixed freely as
 * long as all ranks issue the same sequence.
 *
 * Pushed exchange (the projection and the collective as one kernel):
 * fk_gemm_bf16_push is fk_gemm_bf16 for a row-parallel projection
 * (RowParallelLinear.forward, fastkernels/tasks/baseline/L2/parallel_linear.py:
 * 327-335) whose result is all-reduced next: instead of y, every tile's epilogue
 * stores its outputs straight into the receive areas of ALL ranks over NVLink, as
 * 8-byte {two bf16, call number} words, each written atomically -- the transfer
 * runs tile by tile under the rest of the projection.  dst = HOST array of nranks
 * device addresses, entry r = THIS sender's area inside rank r's buffer
 * ([m][n / 2] words, 16-byte aligned); call_counters = the per-row counters in this
 * rank's own header (buffer + fk_comm_epoch_offset()).
 * fk_allreduce_add_rmsnorm_pushed then reads only local memory: per element it
 * waits (bounded, 2 s) until the nranks senders' words carry this call's number,
 * sums them in rank order and finishes exactly like fk_allreduce_add_rmsnorm (same
 * bits).  One NVLink traversal per call instead of three, at twice the bytes on
 * the wire: fk_allreduce_push_preferred says where that pays (this build: while
 * (nranks - 1) * rows * cols * 4 <= 4 MiB).  Receive areas of one slot lie
 * sender_stride_bytes apart from ll_offset_bytes on; two slots alternate as above.
 *
 * fk_allreduce_add_rmsnorm_group: all nranks ranks in ONE cooperative launch, for
 * a process that holds every rank's buffer on a single device (a test on one GPU,
 * a host emulating shards).  residuals / outs are HOST arrays of nranks device
 * pointers; staging_offset_bytes = 0 selects the one-stage exchange.  Kernels that
 * wait for one another must not be issued as separate launches on one GPU
 * (nothing guarantees they are resident together); the blocks of a cooperative
 * launch are, and the grid is sized to fit (a block walks several rows when
 * rows * nranks exceeds what the device holds at once).  No counterpart in the
 * reference.
 * ---------------------------------------------------------------------- */
size_t fk_comm_header_bytes(void);
int fk_comm_alloc(size_t bytes, void** ptr);
int fk_comm_free(void* ptr);
int fk_comm_ipc_export(void* ptr, void* handle64);
int fk_comm_ipc_import(const void* handle64, void** peer_ptr);
int fk_comm_ipc_close(void* peer_ptr);
int fk_allreduce_add_rmsnorm(void* const* bases, int nranks, int rank,
                             size_t slot_offset_bytes, void* residual,
                             int64_t residual_stride, const void* weight,
                             float eps, void* out, int64_t out_stride,
                             int64_t rows, int64_t cols, int32_t* status,
                             fk_stream_t stream);
int fk_allreduce_two_stage_preferred(int nranks, int64_t rows, int64_t cols);
size_t fk_comm_epoch_offset(void);
int fk_allreduce_push_preferred(int nranks, int64_t rows, int64_t cols);
int fk_gemm_bf16_push(const void* x, int64_t x_stride, const void* w, const void* bias,
                      int64_t m, int64_t n, int64_t k, void* workspace,
                      size_t workspace_bytes, void* const* dst, int nranks,
                      const void* call_counters, int32_t* status, fk_stream_t stream);
int fk_allreduce_add_rmsnorm_pushed(void* base, int nranks, size_t ll_offset_bytes,
                                    size_t sender_stride_bytes, void* residual,
                                    int64_t residual_stride, const void* weight, float eps,
                                    void* out, int64_t out_stride, int64_t rows, int64_t cols,
                                    int32_t* status, fk_stream_t stream);
int fk_allreduce_add_rmsnorm_staged(void* const* bases, int nranks, int rank,
                                    size_t slot_offset_bytes, size_t staging_offset_bytes,
                                    void* residual, int64_t residual_stride,
                                    const void* weight, float eps, void* out,
                                    int64_t out_stride, int64_t rows, int64_t cols,
                                    int32_t* status, fk_stream_t stream);
int fk_allreduce_add_rmsnorm_group(void* const* bases, int nranks,
                                   size_t slot_offset_bytes, size_t staging_offset_bytes,
                                   void* const* residuals, int64_t residual_stride,
                                   const void* weight, float eps, void* const* outs,
                                   int64_t out_stride, int64_t rows, int64_t cols,
                                   int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Fill `count` 32-bit words at dst (16-byte aligned) with `value`: zeroing of
 * workspaces and KV pools on the caller's stream, and the L2 flush of the
 * micro-benchmarks.  No counterpart in the reference (torch.zeros there).
 * ---------------------------------------------------------------------- */
int fk_fill_u32(void* dst, int64_t count, uint32_t value, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * *out ^= XOR of the `count` 32-bit words at src (16-byte aligned, count a
 * multiple of 4; the caller zeroes *out first): a checksum of a workspace or a
 * KV pool on the caller's stream, and the read-only stream the micro-benchmarks
 * time as the read peak of the device.  No counterpart in the reference.
 * ---------------------------------------------------------------------- */
int fk_xor_u32(const void* src, int64_t count, uint32_t* out, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Variable-length prefill attention, the step before decode.
 * Replaces FlashAttnPrefill.forward
 *   (fastkernels/tasks/baseline/L1/flash_attn_prefill.py:28-74; PyTorch
 *   statement Attention._prefill_torch_from_tensors / _prefill_torch_from_cache,
 *   fastkernels/tasks/baseline/L2/attention_impl.py:624-652).
 * For sequence i, query token t (0-based inside the sequence) and head h:
 *   out = softmax(scale * q . K[i, :n]^T) V[i, :n],  n = k_len_i - q_len_i + t + 1
 * when causal (bottom-right aligned, as flash_attn_varlen_func), n = k_len_i
 * otherwise; q_len_i = cu_seqlens_q[i+1] - cu_seqlens_q[i], k_len_i likewise.
 *   q, out   [total_q, Hq, 128] bf16 with token strides (elements)
 *   out_lse  optional fp32 [Hq, total_q]: natural-log sum of exp of the scaled
 *            scores (-inf for a row without visible keys)
 *   K / V    num_blocks == 0: dense [total_k, Hkv, 128], kv_stride = token stride,
 *            sequence i at rows cu_seqlens_k[i] ..;
 *            num_blocks  > 0: the paged pool as in fk_paged_decode_attn
 *            (kv_stride = block stride, block_size, kv_layout), sequence i's
 *            pages in block_tables[i, :]; only the DIFFERENCES of cu_seqlens_k
 *            are used then (flash_attn_prefill.py:41-42)
 *   cu_seqlens_q, cu_seqlens_k  int32 [num_seqs + 1], on the device
 *   max_seqlen_q  upper bound of q_len_i (sizes the grid)
 * head_dim must be 128.  status: optional device word (FK_DEV_BAD_PAGE,
 * FK_DEV_WAIT_TIMEOUT).
 * ---------------------------------------------------------------------- */
int fk_prefill_attn(const void* q, int64_t q_stride_token, void* out,
                    int64_t out_stride_token, float* out_lse, const void* k,
                    const void* v, int64_t kv_stride, int64_t num_blocks,
                    int block_size, int kv_layout, const int32_t* cu_seqlens_q,
                    const int32_t* cu_seqlens_k, const int32_t* block_tables,
                    int64_t block_table_stride, int num_seqs, int64_t total_q,
                    int64_t total_k, int max_seqlen_q, int num_q_heads,
                    int num_kv_heads, int head_dim, float softmax_scale, int causal,
                    int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Merge of two partial attention results over disjoint key ranges.
 * Replaces merge_attn_states / MergeAttnStates.forward
 *   (fastkernels/tasks/baseline/L1/merge_attn_states.py:32-122, kernel
 *   merge_attn_states.cu:2440-2580).
 *   out[t,h,:] = (e^{pl} prefix[t,h,:] + e^{sl} suffix[t,h,:]) / (e^{pl} + e^{sl}),
 *   out_lse[h,t] = log(e^{pl} + e^{sl}),  pl = prefix_lse[h,t], sl = suffix_lse[h,t]
 * computed against max(pl, sl) in fp32, one rounding to bf16.  An lse of +inf
 * counts as -inf; when both are -inf the prefix row is passed through and
 * out_lse = -inf.  Tokens t >= prefill_tokens_with_context (negative = all
 * tokens have context) copy the suffix row and suffix lse.
 *   outputs  [num_tokens, num_heads, head_dim] bf16, token and head strides in
 *            elements; lse fp32 [num_heads, num_tokens]; out_lse optional.
 * ---------------------------------------------------------------------- */
int fk_merge_attn_states(void* out, int64_t out_stride_token, int64_t out_stride_head,
                         float* out_lse, const void* prefix_out,
                         int64_t prefix_stride_token, int64_t prefix_stride_head,
                         const float* prefix_lse, const void* suffix_out,
                         int64_t suffix_stride_token, int64_t suffix_stride_head,
                         const float* suffix_lse, int64_t num_tokens, int num_heads,
                         int head_dim, int64_t prefill_tokens_with_context,
                         fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Decoders with an fp32 residual stream and linear-attention mixers.
 *
 * `is_f32` picks the activation type (0: bf16, 1: fp32); weights of norms, biases
 * and everything that enters the recurrence are fp32 in both.  Rows are padded to
 * `stride` elements with a zero tail.  A batch is a list of portions, each a run of
 * consecutive tokens of one sequence: cu_portions [num_portions + 1] int32 row
 * ranges, slots [rows] int32 = the sequence's state slot (-1: padded row),
 * positions [rows] int64 inside the sequence (0: the state starts at zero).
 * ------------------------------------------------------------------------ */

/* x[i] = float(table[ids[i]]), table [vocab, stride]. */
int fk_embed_f32(const void* table, int is_f32, int64_t vocab, const int64_t* ids, float* x,
                 int64_t rows, int stride, int32_t* status, fk_stream_t stream);

/* x' = x + rms(y) * y_gain (y null: x' = x), stored to x_out when given;
 * h = rms(x') * gain with ONE gain each; out = h + (h_prev - h) * shift with h_prev
 * the sequence's previous h (`state` [num_slots, stride] fp32 across calls, updated),
 * or out = h when shift is null.  With a shift x_out must not be x_in. */
int fk_norm_shift(const float* x_in, float* x_out, const void* y, int64_t y_stride,
                  const float* y_gain, const float* gain, const float* shift, void* out,
                  int is_f32, float* state, int num_slots, const int32_t* slots,
                  const int64_t* positions, const int32_t* cu_portions, int num_portions,
                  int64_t rows, int stride, int width, float eps, int32_t* status,
                  fk_stream_t stream);

/* m = (rms(a) * weight_a + rms(b) * weight_b) / 2; x += rms(m) * gain_out;
 * out = rms(x) * gain (out null: not computed). */
int fk_branch_combine(const void* a, const void* b, int64_t ab_stride, const float* weight_a,
                      const float* weight_b, const float* gain_out, const float* gain, float* x,
                      void* out, int is_f32, int64_t rows, int stride, int width, float eps,
                      fk_stream_t stream);

/* Per head: interleaved rotation (pair 2e, 2e+1) of the first rot_dims channels with
 * cos_sin [max_position, rot_dims] = (cos | sin) fp32, then division by the root mean
 * square over head_dim.  q -> q_out [rows, num_kv_heads * padded_group, padded_dim]
 * (query heads of a KV head padded to padded_group, zeros), k -> k_cache, and k as
 * projected -> v_cache, both NHD [slots, num_kv_heads, padded_dim]. */
int fk_rope_rms_store(const void* q, const void* k, int64_t in_stride, int is_f32, void* q_out,
                      void* k_cache, void* v_cache, const int32_t* slots, int64_t num_slots,
                      const int64_t* positions, const float* cos_sin, int64_t max_position,
                      int rot_dims, int num_q_heads, int num_kv_heads, int head_dim,
                      int padded_group, int padded_dim, float eps, int64_t rows,
                      int32_t* status, fk_stream_t stream);

/* out[i, c] = act(x[i, c]) * x[i, d + c] (act: enum fk_activation). */
int fk_act_and_mul(const void* x, int64_t x_stride, void* out, int64_t out_stride, int is_f32,
                   int64_t rows, int64_t d, int act, fk_stream_t stream);

/* fk_gemm_bf16_silu_mul with a choice of activation; same single-launch shapes. */
int fk_gemm_bf16_act_mul(const void* x, int64_t x_stride, const void* w, const void* bias,
                         void* y, int64_t y_stride, int64_t m, int64_t n, int64_t k, int act,
                         void* workspace, size_t workspace_bytes, int32_t* status,
                         fk_stream_t stream);

/* Generalized delta rule, per head with key channels c and value channels v:
 *   S_t = diag(w_t) S_{t-1} - (a_t * u_t) (u_t^T S_{t-1}) + k_t v_t^T,  o_t = S_t^T r_t
 *   w_t = exp(-decay_scale * sigmoid(w2 tanh(y1) + w0)), a_t = sigmoid(a + a_bias),
 *   u_t = k_t / sqrt(sum k_t^2 + unit_eps)
 * fk_delta_padded_dim: key channels per head in `packed` and `state` (0: unsupported,
 * head size above 256).  fk_delta_prepare writes the operands of the scan from packed
 * projection rows; w2 [heads * dim, w2_stride] in the activation type, rows zero-padded
 * to a multiple of 4 (rank <= 512).  blocked 0: per token, packed
 * [heads][rows][6][padded_dim] fp32 (w, u, a * u, k, r, v), for single tokens;
 * blocked 1: blocks of 8 tokens of a portion (layout: csrc/fk_delta.cu), for portions.
 * fk_delta_packed_floats: size of `packed` in floats.
 * fk_delta_scan runs the recurrence for every portion from and to
 * state [num_slots][heads][dim (value)][padded_dim (key)] fp32 and writes
 * o [rows, heads * dim] fp32.  fk_head_norm_gate: out = rms(o per head) * weight *
 * sigmoid(gate), columns beyond heads * dim zeroed. */
int fk_delta_padded_dim(int dim);
int64_t fk_delta_packed_floats(int64_t rows, int num_portions, int heads, int dim, int blocked);
int fk_delta_prepare(const void* r, const void* k, const void* v, const void* a, const void* y1,
                     int64_t in_stride, int is_f32, const void* w2, int64_t w2_stride,
                     const float* w0, const float* a_bias, float* packed, int blocked,
                     const int32_t* cu_portions, int num_portions, int64_t rows,
                     int heads, int dim, int rank, float decay_scale, float unit_eps,
                     fk_stream_t stream);
int fk_delta_scan(const float* packed, int blocked, float* o, float* state, int num_slots,
                  const int32_t* cu_portions, int num_portions, const int32_t* slots,
                  const int64_t* positions, int64_t rows, int heads, int dim, int32_t* status,
                  fk_stream_t stream);
int fk_head_norm_gate(const float* o, const void* gate, int64_t gate_stride, const float* weight,
                    void* out, int64_t out_stride, int is_f32, int64_t rows, int heads, int dim,
                    float eps, fk_stream_t stream);

/* y[m, n] = x[m, k] w[n, k]^T (+ bias) in fp32 (no tensor cores); k % 4 == 0. */
int fk_gemm_f32(const float* x, int64_t x_stride, const float* w, const float* bias, float* y,
                int64_t y_stride, int64_t m, int64_t n, int64_t k, fk_stream_t stream);

/* Causal attention over the NHD pool for any head size up to 1152 (multiple of 4), any
 * query / KV head ratio, bf16 or fp32: sequence i brings query rows cu_seqlens_q[i] ..
 * cu_seqlens_q[i + 1] that end at its kv_lens[i]-th key. */
int fk_paged_attn_any(const void* q, int64_t q_stride, void* out, int64_t out_stride,
                      const void* k_cache, const void* v_cache, int is_f32, int64_t num_blocks,
                      int block_size, const int32_t* cu_seqlens_q, const int32_t* kv_lens,
                      const int32_t* block_tables, int64_t block_table_stride, int num_seqs,
                      int64_t rows, int num_q_heads, int num_kv_heads, int head_dim,
                      float softmax_scale, int32_t* status, fk_stream_t stream);

/* fk_paged_decode_attn (planned 0) / _planned (planned 1) and fk_prefill_attn with the
 * fp32 softmax weights taken into P V as two bf16 parts (16 significant bits) instead of
 * being rounded to one.  out_head_dim: channels stored per head of out, whose heads lie
 * that far apart (a multiple of 8, at most head_dim). */
int fk_paged_decode_attn_2p(int planned, const void* q, int64_t q_stride_token, void* out,
                            int64_t out_stride_token, const void* k_cache, const void* v_cache,
                            int64_t num_blocks, int block_size, int64_t kv_block_stride,
                            int kv_layout, const int32_t* context_lens,
                            const int32_t* block_tables, int64_t block_table_stride, int batch,
                            int num_q_heads, int num_kv_heads, int head_dim,
                            float softmax_scale, int max_splits, void* workspace,
                            size_t workspace_bytes, int32_t* status, fk_stream_t stream);
int fk_prefill_attn_2p(const void* q, int64_t q_stride_token, void* out,
                       int64_t out_stride_token, float* out_lse, const void* k, const void* v,
                       int64_t kv_stride, int64_t num_blocks, int block_size, int kv_layout,
                       const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                       const int32_t* block_tables, int64_t block_table_stride, int num_seqs,
                       int64_t total_q, int64_t total_k, int max_seqlen_q, int num_q_heads,
                       int num_kv_heads, int head_dim, int out_head_dim, float softmax_scale,
                       int causal, int32_t* status, fk_stream_t stream);

/* ------------------------------------------------------------------------
 * Decoders whose mixer and feed-forward read the same residual row side by side, with
 * latent attention, a matrix memory and mixtures of experts (conventions as above).
 * ------------------------------------------------------------------------ */

/* fk_embed_f32 plus a row of a second table: (previous token * mul_prev + token * mul_cur)
 * mod buckets, row `buckets` for a sequence's first token.  last_ids [num_slots] int64 is
 * each sequence's last token across calls (read and replaced).  pairs null: no second
 * table.  copy (may be null): the row in the activation type as well. */
int fk_embed_pair_f32(const void* table, const void* pairs, int is_f32, int64_t vocab,
                      int64_t buckets, int64_t mul_prev, int64_t mul_cur, const int64_t* ids,
                      int64_t* last_ids, int num_slots, const int32_t* slots,
                      const int64_t* positions, const int32_t* cu_portions, int num_portions,
                      float* x, void* copy, int64_t copy_stride, int64_t rows, int stride,
                      int32_t* status, fk_stream_t stream);

/* x' = x + a + b + sum_j share[t, j] * experts[place[t, j]] (each optional), stored to x_out
 * when given (may be x_in); out1 = layernorm(x') * weight1 + bias1 and, when given, out2
 * alike from the same statistics.  weight1 null: out1 = x'.  expert_rows bounds place. */
int fk_add_layernorm(const float* x_in, float* x_out, const void* a, int64_t a_stride,
                     const void* b, int64_t b_stride, const void* experts, int64_t expert_stride,
                     int64_t expert_rows, const int32_t* place, const float* share, int top,
                     const float* weight1, const float* bias1, void* out1, int64_t out1_stride,
                     const float* weight2, const float* bias2, void* out2, int64_t out2_stride,
                     int is_f32, int64_t rows, int stride, int width, float eps,
                     int32_t* status, fk_stream_t stream);

/* x = cap * tanh(x / cap) in place. */
int fk_softcap(void* x, int64_t stride, int is_f32, int64_t rows, int64_t cols, float cap,
               fk_stream_t stream);

/* Grouped projection y = x w_g^T (+ bias), w [groups][w rows][k].
 *   column groups (offsets null): group g takes all `rows` rows, x columns from g * x_group
 *     and y columns from g * y_group on
 *   row groups: group g takes rows offsets[g] .. offsets[g + 1] (device int32
 *     [groups + 1]) of y; x rows the same, or gather[row]
 * act >= 0 (enum fk_activation): w_g has 2 n rows [gate; up], y = act(gate) * up.  is_f32:
 * fp32 operands and result; else bf16 operands, fp32 accumulation, result bf16 or (y_f32)
 * fp32.  bias fp32, one per row of w_g, the same for all groups.  expect_rows: rows a group has, roughly;
 * picks the kernel. */
int fk_group_gemm(const void* x, int64_t x_stride, int64_t x_group, int64_t x_rows,
                  const void* w, const float* bias, void* y, int64_t y_stride, int64_t y_group,
                  int is_f32, int y_f32, const int32_t* offsets, const int32_t* gather,
                  int64_t rows, int64_t expect_rows, int groups, int64_t n, int64_t k, int act,
                  int32_t* status, fk_stream_t stream);

/* The `top` largest of every row of logits z [rows, experts] (lowest index on ties): chosen
 * and their softmax weights share [rows, top]; place [rows, top] = position of each pair in
 * the list sorted by expert, source [rows * top] = row of every list entry, offsets
 * [experts + 1] = first entry of every expert.  counts: fk_moe_route_counts() int32 of
 * scratch (0: none needed). */
int64_t fk_moe_route_counts(int64_t rows, int experts, int top);
int fk_moe_route(const float* z, int64_t z_stride, int32_t* chosen, float* share, int32_t* place,
                 int32_t* source, int32_t* offsets, int32_t* counts, int64_t rows, int experts,
                 int top, fk_stream_t stream);

/* y[r] = x[source[r]], rows of row_bytes bytes. */
int fk_gather_rows(const void* x, int64_t x_stride_bytes, int64_t x_rows, const int32_t* source,
                   void* y, int64_t rows, int64_t row_bytes, int32_t* status,
                   fk_stream_t stream);

/* Latent attention.  A cached row is [rms(latent) * weight (rank) | rotated key (rot) | 0].
 * fk_latent_prepare: from packed rows, heads of q [dim unrotated | rot] q_pitch apart and
 * latent [rank | rot], store the cached row at its slot and write the rotated part of every
 * query head to q_out [rows, heads, q_out_pitch] from column q_rot_at on (zeros behind it),
 * with copy also the unrotated part from column 0 on.  Rotation interleaved, cos_sin
 * [max_position, rot] = (cos | sin).
 * fk_latent_gather: cached rows of all sequences side by side, cu_seqlens_k [num_seqs + 1].
 * fk_latent_attn (bf16): every (token, head) row of q attends the cached rows of its
 * sequence up to its own token (queries end at key kv_lens[i]); the value of a key is its
 * first `rank` channels; out [rows * heads, out_pitch].  splits > 1 cuts the keys of every
 * row into that many ranges and merges them (fk_latent_attn_splits suggests a number).
 * Rows that do not fit on an SM (fk_latent_attn_supported: rank up to 512) go through
 * fk_paged_attn_any with one KV head. */
int fk_latent_prepare(const void* q, const void* latent, int64_t in_stride, int q_pitch,
                      int is_f32, const float* weight, const float* cos_sin, int64_t max_position,
                      const int32_t* slots, const int64_t* positions, void* cache,
                      int64_t num_slots, int cache_pitch, void* q_out, int q_out_pitch,
                      int q_rot_at, int copy, int64_t rows, int heads, int dim, int rot, int rank,
                      float eps, int32_t* status, fk_stream_t stream);
int fk_latent_gather(const void* cache, int64_t row_bytes, int64_t num_blocks, int block_size,
                     const int32_t* block_tables, int64_t block_table_stride,
                     const int32_t* cu_seqlens_k, int num_seqs, void* out, int64_t rows,
                     int32_t* status, fk_stream_t stream);
int fk_latent_attn_supported(int rank, int rot);
int fk_latent_attn_splits(int num_seqs, int64_t max_q, int heads, int rank, int64_t max_keys);
int64_t fk_latent_attn_workspace_floats(int64_t rows, int heads, int rank, int splits);
int fk_latent_attn(const void* q, int64_t q_pitch, const void* cache, int64_t num_blocks,
                   int block_size, int cache_pitch, void* out, int64_t out_pitch,
                   const int32_t* cu_seqlens_q, const int32_t* kv_lens,
                   const int32_t* block_tables, int64_t block_table_stride, int num_seqs,
                   int64_t rows, int64_t max_seqlen_q, int heads, int rank, int rot,
                   float softmax_scale, int splits, float* workspace, int64_t workspace_floats,
                   int32_t* status, fk_stream_t stream);

/* Matrix memory, per head (equations: csrc/fk_mlstm.cu).  q, k [rows, heads * dim] and
 * v [rows, heads * vdim] are columns of packed rows; z fp32 [rows, 2 * heads] holds the
 * pre-activations of the input and of the forget gates.  State of a sequence: s_state
 * [num_slots, heads, dim, fk_mlstm_state_cols(vdim)], n_state [num_slots, heads,
 * fk_mlstm_norm_cols(dim)], fp32, read and replaced; zero at position 0.
 * fk_mlstm_step: one token per row, out = rms(o per head) * weight * sigmoid(gate).
 * fk_mlstm_portions: runs of tokens, o fp32 [rows, heads * vdim] before norm and gate.  With
 * a workspace (fk_mlstm_workspace_floats) bf16 portions go 128 tokens at a time, without one
 * token by token.  longest: tokens of the longest portion. */
int fk_mlstm_state_cols(int vdim);
int fk_mlstm_norm_cols(int dim);
int fk_mlstm_step(const void* q, const void* k, const void* v, int64_t in_stride, int is_f32,
                  const float* z, int64_t z_stride, const void* gate, int64_t gate_stride,
                  const float* weight, float* s_state, float* n_state, int num_slots,
                  const int32_t* slots, const int64_t* positions, void* out, int64_t out_stride,
                  int64_t rows, int heads, int dim, int vdim, float gate_cap, float q_scale,
                  float eps, int32_t* status, fk_stream_t stream);
int64_t fk_mlstm_workspace_floats(int64_t rows, int num_portions, int heads, int dim, int vdim);
int fk_mlstm_portions(const void* q, const void* k, const void* v, int64_t in_stride, int is_f32,
                      const float* z, int64_t z_stride, float* s_state, float* n_state,
                      int num_slots, const int32_t* cu_portions, int num_portions,
                      const int32_t* slots, const int64_t* positions, float* o, int64_t rows,
                      int heads, int dim, int vdim, float gate_cap, float q_scale,
                      float* workspace, int64_t workspace_floats, int64_t longest,
                      int32_t* status, fk_stream_t stream);

/* fk_argmax_bf16 on fp32 rows. */
int fk_argmax_f32(const float* x, int64_t x_stride, int64_t rows, int64_t cols, float* out_val,
                  int64_t* out_idx, fk_stream_t stream);

#ifdef __cplusplus
}
#endif

#endif /* FK_B200_H_ */
