// C ABI of libnanoflow_kernels.so. Every entry point takes raw device pointers and a CUDA stream,
// launches asynchronously on that stream, allocates nothing, and returns 0 on success or one of
// the NF_ERR_* codes (common.cuh) when an argument is rejected before any launch.
// bf16 tensors are passed as void*; int tensors are int32 unless noted.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

// ------------------------------------------------------------------------------------------------
// GEMM (gemm.cu)
// ------------------------------------------------------------------------------------------------
enum { NFK_EPI_LINEAR = 0, NFK_EPI_SWIGLU = 1, NFK_EPI_REDUCE_SCATTER = 2 };
// Gated epilogue: act(gate) * up, or for NFK_ACT_CAPPED g sigmoid(alpha g) (u + shift) with g = min(gate, limit) and
// u = min(max(up, -limit), limit).
enum { NFK_ACT_SILU = 0, NFK_ACT_RELU = 1, NFK_ACT_GELU_TANH = 2, NFK_ACT_CAPPED = 3 };
// activation of the linear epilogue (GELU: by erf; RELU2: the square of relu)
enum { NFK_LIN_NONE = 0, NFK_LIN_TANH = 1, NFK_LIN_GELU = 2, NFK_LIN_RELU2 = 3 };
enum { NFK_BF16 = 0, NFK_F32 = 1 };                                    // storage type of activations and weights

typedef struct nfk_gemm_params {
  const void* A;    // [M,K] bf16, row-major, leading dimension lda
  const void* B;    // [N,K] bf16, row-major (nn.Linear weight layout); gate weight for SwiGLU
  const void* B2;   // SwiGLU only: up weight [N,K]
  void* D;          // [M,N] bf16
  const void* C;    // optional residual [M,N]: D = A*B^T + bias + beta*C
  const void* bias; // optional [N] bf16
  long long lda, ldb, ldd, ldc;
  float beta;
  int M, N, K;
  int epilogue;     // NFK_EPI_*
  int tile_n;       // 0 = choose; tile width in weight rows: a multiple of 32 up to 256
  int num_ctas;     // CTA budget of the persistent grid; 0 = one per SM
  unsigned int* status;  // optional device word: first non-zero NF_ST_* code wins
  int tile_m;       // 0 = choose; number of 128-row M tiles one CTA covers: 1 / 2 / 4
  int split_k;      // 0 = choose; > 1 needs `workspace` (fp32 partials, split_k*M*N*4 bytes)
  void* workspace;  // scratch for fp32 partial sums (split-K, stream-K tail); GEMMs that may overlap need their own
  long long workspace_bytes;
  // NFK_EPI_REDUCE_SCATTER: the epilogue does not write D; it pushes every bf16 partial row straight
  // into the slab of the rank that owns the row (row i belongs to rank i % rs_nranks), over NVLink:
  //   heap[owner] + rs_slab_off + ((rs_rank * rs_rows_cap + i / rs_nranks) * N + col) * 2
  // and, once all CTAs are done, raises ready[rs_rank] = rs_epoch in the flag block at rs_flag_off
  // on every rank. nfk_allreduce with src_mode 1 then reduces the slabs locally.
  void* rs_heap[8];
  int rs_rank, rs_nranks;
  long long rs_slab_off;
  int rs_rows_cap;
  long long rs_flag_off;
  int rs_epoch;
  int smem_budget_kb;  // 0 = all 227 KB; smaller leaves shared memory for a kernel meant to share the SM
  int cta_group;       // 0 = let the cost model decide; 1 = one CTA per tile; 2 = a CTA pair per 256-row tile
  int stream_k;        // tail wave cut into k ranges: 0 = cost model (off when the tile shape is pinned), 1 = on, 2 = off,
                       // 3 = off and one work unit per CTA, dealt out by the hardware block scheduler (for a GEMM
                       // that shares SMs with another stream's kernel)
  // Optional RMSNorm of the result rows: norm_out[M, N] = RMSNorm(D) * norm_w (what the next layer's
  // first GEMM reads). With split-K the reduce pass produces it from the rows it already holds;
  // otherwise the launcher adds a norm launch after the GEMM. Linear epilogue only.
  const void* norm_w;   // [N] bf16, null = no norm
  void* norm_out;       // [M, norm_ld] bf16
  long long norm_ld;
  float norm_eps;
  // Reduce-scatter epilogue: 1 = rows leave through a shared-memory staging piece and one bulk copy per
  // row and 128 columns (256-byte NVLink writes); 0 = 16-byte stores straight from registers.
  int rs_staged;
  // Gated input (all-gather -> GEMM in one pipeline): the rows of A are still being delivered by a
  // collective when the GEMM starts. gate_flags points to this GPU's copy of the collective's row-block
  // flags, [ceil(M/128)][8] words: word [b][r] reaches gate_epoch once rank r has delivered all of its rows
  // of block b (rows 128b .. 128b+127). The TMA producer of a CTA waits (bounded) for the gate_nranks words
  // of an M tile before its first load of that tile, and tiles are walked row block by row block (all
  // column blocks of the first rows first), so the main loops of the first tiles run while the collective
  // is still delivering the later rows. Null = A is complete before the launch. Linear and SwiGLU
  // epilogues; no split-K and no stream-K tail in this mode.
  const unsigned int* gate_flags;
  int gate_epoch, gate_nranks;
  // Linear epilogue: output columns from f32_col0 on are written as fp32 to D32[row * ld32 + col - f32_col0]
  // instead of bf16 to D (f32_col0 0: all of them, D may be null). Null = none.
  void* D32;
  long long ld32;
  int f32_col0;         // multiple of 8
  int act;              // gated epilogue: NFK_ACT_*
  // Block-diagonal product (linear epilogue): `groups` > 1 cuts the N columns (and B's rows) into equal
  // groups; group g reads A's columns [g * group_k, g * group_k + K). 0 or 1 = an ordinary product.
  int groups, group_k;
  int lin_act;          // linear epilogue: NFK_LIN_*, applied to the finished columns
  float act_limit, act_alpha, act_shift;   // constants of NFK_ACT_CAPPED
  const void* bias2;    // gated epilogue: [N] bf16 bias of the up half (`bias` is the gate half's), null = none
} nfk_gemm_params;

int nfk_gemm_bf16(const nfk_gemm_params* p, cudaStream_t stream);
// The same products with fp32 operands and outputs in fp32 FMA arithmetic (gemm_f32.cu): A, B, B2, D, C, bias
// are fp32, D32 as above; tile / split / budget / gate fields are ignored, norm and reduce-scatter not built.
int nfk_gemm_f32(const nfk_gemm_params* p, cudaStream_t stream);

typedef struct nfk_gemm_plan {
  int tile_n, tile_m, cta_group, split_k, stream_k;
  int tiles, workers, num_kb;          // output tiles, CTAs (or CTA pairs), 64-wide k-blocks
  int tail_first_tile, tail_range_kb, tail_max_pieces;   // stream-K tail (tail_range_kb 0 = none)
  int stages, smem_bytes;
} nfk_gemm_plan;
int nfk_gemm_describe(const nfk_gemm_params* p, nfk_gemm_plan* out);

// ------------------------------------------------------------------------------------------------
// Elementwise / normalisation / gather kernels (elementwise.cu)
// ------------------------------------------------------------------------------------------------
// out[r,:] = x[r,:] * rsqrt(mean(x[r,:]^2) + eps) * w[:]
int nfk_rmsnorm(void* out, const void* x, const void* w, int rows, int cols, float eps,
                cudaStream_t stream);
// resid[r,:] += x[r,:]; out[r,:] = rmsnorm(resid[r,:]) (resid updated in place)
int nfk_add_rmsnorm(void* out, void* resid, const void* x, const void* w, int rows, int cols,
                    float eps, cudaStream_t stream);
// Token ids for this iteration, then the embedding rows:
//   id[t] = feedback_src[t] >= 0 ? prev_tokens[feedback_src[t]] : host_ids[t]
//   out[t,:] = table[id[t],:]      (ids outside [0,vocab) are clamped and flagged in status)
// feedback_src / prev_tokens may be null (ids come from host_ids only). ids_out may be null.
int nfk_embedding(void* out, const void* table, const int* host_ids, const int* feedback_src,
                  const int* prev_tokens, int* ids_out, int n_tokens, int hidden, int vocab,
                  unsigned int* status, cudaStream_t stream);
// out[i,:] = in[rows_idx[i],:]
int nfk_gather_rows(void* out, const void* in, const int* rows_idx, int n, int cols, long long ld_in,
                    unsigned int* status, int in_rows, cudaStream_t stream);
// out = silu(gate) * up, elementwise over n elements (n % 8 == 0)
int nfk_silu_mul(void* out, const void* gate, const void* up, long long n, cudaStream_t stream);
// out[r, 0:cols] = in[r, col0 : col0+cols]   (column-block extract / insert with leading dims)
int nfk_copy_cols(void* out, long long ld_out, const void* in, long long ld_in, int rows, int cols,
                  cudaStream_t stream);
// 2-D transpose out[c,r] = in[r,c]
int nfk_transpose(void* out, const void* in, int rows, int cols, cudaStream_t stream);
// Greedy sampler: per row arg-max over `cols` logits. idx_out[r] = col_offset + argmax,
// val_out[r] (optional, fp32) = max. Ties resolve to the lowest index.
int nfk_argmax(int* idx_out, float* val_out, const void* logits, int rows, int cols,
               long long ld, int col_offset, cudaStream_t stream);
// The same over fp32 logits.
int nfk_argmax_f32(int* idx_out, float* val_out, const float* logits, int rows, int cols, long long ld,
                   int col_offset, cudaStream_t stream);
// Combine per-shard (val, idx) candidates: cand_val/cand_idx are [shards, rows].
int nfk_argmax_combine(int* idx_out, const float* cand_val, const int* cand_idx, int shards,
                       int rows, cudaStream_t stream);
// Busy-wait for `micros` microseconds (bounded at 1 s); stands in for a collective in ablations.
int nfk_sleep(int micros, cudaStream_t stream);
// Device progress counters: add / clear / bounded wait until *flag >= target.
int nfk_flag_add(unsigned int* flag, unsigned int v, cudaStream_t stream);
int nfk_flag_clear(unsigned int* flag, cudaStream_t stream);
int nfk_flag_wait(const unsigned int* flag, unsigned int target, int timeout_us,
                  unsigned int* status, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// RoPE + paged-KV append (rope_append.cu)
// ------------------------------------------------------------------------------------------------
// Paged KV pool of one layer: [num_pages][2 (K,V)][kv_heads][page_size][head_dim] bf16.
typedef struct nfk_rope_append_params {
  const void* qkv;       // [T, ld_qkv] bf16: q at q_off, k at k_off, v at v_off (elements)
  long long ld_qkv;
  int q_off, k_off, v_off;
  void* q_out;           // [T, q_heads*head_dim] rotated queries
  void* kv_pool;         // this layer's pool
  const float* inv_freq; // [head_dim/2] rotary inverse frequencies (any scaling baked in)
  const int* positions;  // [T] absolute position of each token in its sequence
  const int* token_req;  // [T] request index of each token
  const int* kv_indptr;  // [B+1]
  const int* kv_indices; // page ids
  int T, q_heads, kv_heads, head_dim, page_size, num_pages;
  unsigned int* status;
  const float* cos_sin;  // optional [T][head_dim/2][2] (cos, sin) of every token's angles (nfk_rope_table);
                         // null: the kernel computes them itself
} nfk_rope_append_params;
int nfk_rope_append(const nfk_rope_append_params* p, cudaStream_t stream);

// cos / sin of pos[t] * inv_freq[i] for the T tokens of an iteration: every layer rotates by the same
// angles, so they are computed once per iteration instead of once per layer.
typedef struct nfk_rope_table_params {
  float* cos_sin;        // out [T][half][2]
  const float* inv_freq; // [half]
  const int* positions;  // [T]
  int T, half;
} nfk_rope_table_params;
int nfk_rope_table(const nfk_rope_table_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Attention over the paged KV pool (attention.cu)
// ------------------------------------------------------------------------------------------------
typedef struct nfk_attn_params {
  const void* q;           // [T, q_heads*head_dim] bf16 (rotated)
  void* out;               // [T, q_heads*head_dim] bf16
  const void* kv_pool;     // layer pool, layout above
  const int* qo_indptr;    // [B+1] token range of every request in the dense batch
  const int* kv_indptr;    // [B+1]
  const int* kv_indices;
  const int* kv_last_page_len;  // [B]
  int q_heads, kv_heads, head_dim, page_size, num_pages;
  float sm_scale;
  int num_ctas;            // CTA budget (persistent grid); 0 = one per SM
  // decode: requests [req_begin, req_begin+req_count) each own one query token (qo_indptr[b])
  int req_begin, req_count;
  int chunk_pages;         // split-KV chunk length in pages; 0 = no split
  float* workspace;        // split-KV partials: [req_count*q_heads*max_chunks*(head_dim+2)] fp32
  int max_chunks;
  // prefill: work items (req, first token (global index), token count)
  const int* items;        // [num_items,3]
  int num_items;
  unsigned int* status;
  int decode_stages;       // decode: pages in flight per warp, 3 (0 means 3) or 2 (less shared memory per CTA)
  // nfk_attn_prefill_ws only:
  int window;              // > 0: position i sees j with 0 <= i - j < window
  const float* sinks;      // [q_heads]: exp(sink) joins the softmax denominator; null = none
  // kv_ld > 0: keys and values are not pool pages but columns of plain rows: page id x stands for rows
  // 16 x .. 16 x + 15 of a [num_pages * 16][kv_ld] array, head h's key at column k_col + 128 h, value at v_col + 128 h
  int kv_ld, k_col, v_col;
  int q_rows;              // > 0 (one query head per KV head): rows of q, which is [q_rows][ld_q]
  int ld_q;                // 0 = q_heads * 128
  // nfk_attn_decode and nfk_attn_prefill_ws (head_dim 64 or 128):
  float softcap;           // > 0: score <- softcap tanh(score / softcap) before the softmax
  int precise;             // 1: probabilities enter the second product as a bf16 pair (implied by the other extensions)
  // nfk_attn_decode and nfk_attn_prefill_ws, together with `precise`. ld_q (elements from token to token of q, a multiple of
  // head_dim) also holds for these.
  const int* kv_first;     // [B] page slot of the sequence that a request's page list starts with; null = 0
  const float* dist;       // [q_heads][2] (a, b): score <- score - a ln(1 + b (i - j)); null = none
  int chunk;               // > 0: position i sees j only if i / chunk = j / chunk
} nfk_attn_params;
int nfk_attn_decode(const nfk_attn_params* p, cudaStream_t stream);
// The same with the pages copied by a TMA producer warp into a ring of decode_stages (2, 3 or 4) pages per
// consumer warp, one work item per warp (attention_dec.cu): full bandwidth from one CTA per SM, for sharing
// SMs with GEMM CTAs. head_dim 128; calls with chunk_pages > 0 are forwarded to nfk_attn_decode.
int nfk_attn_decode_tma(const nfk_attn_params* p, cudaStream_t stream);
int nfk_attn_prefill(const nfk_attn_params* p, cudaStream_t stream);
// Same contract as nfk_attn_prefill for head_dim 128, on tcgen05 tensor cores (attention_tc.cu).
int nfk_attn_prefill_tc(const nfk_attn_params* p, cudaStream_t stream);
// The same on a warp-specialised pipeline: a TMA load warp (whole pages, no transposes), an MMA warp that
// issues the next tile's scores under this tile's softmax, four softmax warps (attention_ws.cu).
int nfk_attn_prefill_ws(const nfk_attn_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Layer-list models: residual step, latent attention, mLSTM (residual_norm.cu, latent.cu, mlstm.cu)
// ------------------------------------------------------------------------------------------------
enum { NFK_NORM_NONE = 0, NFK_NORM_RMS = 1, NFK_NORM_LAYER = 2, NFK_NORM_SCALE = 3 };   // SCALE: only times the weights
// x <- (table ? 0 : x) + norm_in(src_scale src) (+ y2_gate y2) (+ sum_k e_weight e_out[e_slot]) (+ add);  h = norm_out(x).
// norm_sum: norm_in takes in y2 and the experts' rows too. pair_w: the source is half the sum of RMS norms of y (times
// pair_w) and y2 (times pair_w2). table_add: x <- x + ... + src_scale (embedding row), which is then not a source.
// pos_freq: a sinusoidal position vector joins the embedding row, entry 2i sin(p f_i), entry 2i + 1 cos(p f_i).
// hist: earlier versions of the stream. The sum goes to hist_out; with hist_w, x <- hist_w[hist_n] (sum) + sum_j hist_w[j]
// hist[j] is what goes on.
// Rows of x, y, table and h are padded to a multiple of 4 elements; weight vectors are padded with zeros to that length.
typedef struct nfk_residual_norm_params {
  float* x;                  // [*, ld_x] residual stream
  long long ld_x;
  const void* y;             // [*, ld_y] sublayer output, null: none
  long long ld_y;
  const void* table;         // [vocab, ld_table] embedding: the source is the token's row instead of y
  long long ld_table;
  const int* host_ids;       // token ids as in nfk_embedding
  const int* feedback_src;
  const int* prev_tokens;
  int vocab;
  const float* in_w;         // norm of the source
  const float* in_b;
  const float* add;          // [cols] added to the stream after the sum, null: none
  void* h;                   // [rows, ld_h] normed stream for the next sublayer, null: none
  long long ld_h;
  const float* out_w;
  const float* out_b;
  const int* rows_idx;       // row r of h comes from row rows_idx[r] of x and y; x is not written back then
  int in_rows;
  int rows, cols;
  float eps;
  int in_kind, out_kind;     // NFK_NORM_*
  int dtype;                 // NFK_BF16 / NFK_F32: y, table, h, y2, e_out
  unsigned int* status;
  float src_scale;           // factor of the source row; 0 = 1
  const void* y2;            // [*, ld_y2] a second sublayer output that joins the same sum, null: none
  long long ld_y2;
  const float* y2_gate;      // [*] factor per row of y2, null: 1
  const void* e_out;         // [e_rows, ld_e] outputs of a mixture of experts, null: none
  long long ld_e;
  const int* e_slot;         // [*][e_top] rows of e_out of a token, -1: none
  const float* e_weight;     // [*][e_top]
  int e_top, e_rows;
  int norm_sum;
  const float* pair_w;       // [cols] padded, null: none
  const float* pair_w2;
  int table_add;
  // Input convolution of the next sublayer (see nfk_short_conv, residual form) for the first conv_rows rows, each the only
  // token of the request of the same number: the result goes to conv_out instead of h's row.
  const float* conv_w;       // [conv_taps][conv_ld], null: none
  void* conv_out;            // [*, conv_ld]
  void* conv_state;          // [slots][2][max(1, conv_taps - 1)][conv_ld]
  const int* state_slot;
  const int* positions;
  int conv_taps, conv_rows, conv_ld, num_slots;
  const float* pos_freq;     // [(cols + 1) / 2][2]: f_i as the sum of two floats, null: none; needs positions
  const float* hist;         // [hist_n][*, ld_x], hist_stride elements apart
  const float* hist_w;       // [hist_n + 1], null: none
  float* hist_out;           // [*, ld_x], null: none
  long long hist_stride;
  int hist_n;
} nfk_residual_norm_params;
int nfk_residual_norm(const nfk_residual_norm_params* p, cudaStream_t stream);

// Latent pool of one layer: pages of page_size rows of ld elements (ld = latent size padded to a multiple of 8, the
// padding is zero). bf16 pages whose ld is a multiple of 64 are stored in tiles, [page_size / 8][ld / 64][8 rows][64
// columns], so that one TMA copy brings in a whole page in the layout the tensor cores read; all others row by
// row. Token t's latent: RMS norm of src[t, 0:rank] times w, written to its page slot.
// kv_first[req]: page slot of the sequence that the request's page list starts with (null: 0).
typedef struct nfk_latent_append_params {
  const void* src;
  long long ld_src;
  const float* w;
  void* pool;
  long long ld;
  const int* positions;
  const int* token_req;
  const int* kv_indptr;
  const int* kv_indices;
  const int* kv_first;
  int T, rank, page_size, num_pages;
  float eps;
  int dtype;
  unsigned int* status;
} nfk_latent_append_params;
int nfk_latent_append(const nfk_latent_append_params* p, cudaStream_t stream);

// Pages of a latent pool -> plain rows: out[i * page_size + r, :] = row r of page page_ids[i].
typedef struct nfk_latent_gather_params {
  const void* pool;
  void* out;                 // [n_pages * page_size, ld]
  const int* page_ids;
  long long ld;
  int n_pages, page_size, num_pages, dtype;
  unsigned int* status;
} nfk_latent_gather_params;
int nfk_latent_gather(const nfk_latent_gather_params* p, cudaStream_t stream);

// Attention in latent space, for listed tokens: head h's query (already multiplied by its key matrix) meets
// the cached latents, which are keys and values at once: out = sum_j softmax(scale q . c_j) c_j over the
// positions i - window < j <= i (window 0: all j <= i), with exp(sink[h]) in the denominator (sinks null: none).
typedef struct nfk_latent_attn_params {
  const void* q;             // [*, ld_q]: head h of a token at column h * ld
  long long ld_q;
  const void* pool;
  long long ld;              // padded latent size
  void* out;                 // [*, ld_out]: head h at column h * ld
  long long ld_out;
  const int* tokens;         // [n_tokens] token rows
  const int* positions;
  const int* token_req;
  const int* kv_indptr;
  const int* kv_indices;
  const int* kv_first;
  const float* sinks;        // [heads]
  int n_tokens, heads, page_size, num_pages, window;
  float scale;
  int dtype;
  int impl;                  // 0 = choose, 1 = simple kernel, 2 = tensor-core kernel (bf16)
  int splits;                // tensor-core kernel: key ranges per token, > 1 needs a workspace
  float* workspace;          // [n_tokens][splits][heads][ld + 2] fp32
  long long workspace_floats;
  unsigned int* status;
} nfk_latent_attn_params;
int nfk_latent_attn(const nfk_latent_attn_params* p, cudaStream_t stream);

// mLSTM. Per request slot and head: S [dim][vdim], n [2][dim], m [2], fp32. A launch reads one half of n and m
// and writes the other, so that CTAs which share a head (each owns columns of S) can all read the old ones
// while one of them writes the new ones; the caller flips the half with every step of the request. A request
// whose first token of the launch is at position 0 starts from zero.
typedef struct nfk_mlstm_params {
  const void* qkv;           // [T, ld_qkv]: q at q_off + h * dim, k at k_off, v at v_off + h * vdim
  long long ld_qkv;
  int q_off, k_off, v_off;
  const float* gates;        // [T, ld_gates]: input gate of head h at column h, forget gate at heads + h
  long long ld_gates;
  const float* i_bias;       // [heads]
  const float* f_bias;
  float* S;                  // [slots][heads][dim][vdim]
  float* n;                  // [slots][heads][2][dim]
  float* m;                  // [slots][heads][2]
  float* out;                // [T, ld_out]: head h at column h * vdim
  long long ld_out;
  const int* positions;
  const int* qo_indptr;
  const int* state_slot;     // [B] 2 * slot + half of n / m to read
  int req_begin, req_count;
  int heads, dim, vdim;      // dim, vdim: padded to multiples of 8 (padding columns are zero)
  int num_slots;
  float gate_cap, q_scale;
  int dtype;
  int impl;                  // prefill: 0 = choose, 1 = token by token, 2 = chunked on tensor cores (bf16)
  // chunked form: items [num_items][4] (request, first token, tokens, segment of the request), in token order, and
  // scratch: (num_tokens / 64 + num_items + 1) * heads * 192 floats of gate values, and if a request has several
  // segments num_items * heads * (dim * vdim + dim + 8) floats for their states
  const int* items;
  int num_items;
  int num_tokens;            // rows of qkv that hold tokens of this iteration
  float* scratch;
  long long scratch_floats;
  unsigned int* status;
} nfk_mlstm_params;
int nfk_mlstm_decode(const nfk_mlstm_params* p, cudaStream_t stream);    // one token per request
int nfk_mlstm_prefill(const nfk_mlstm_params* p, cudaStream_t stream);   // any number of tokens per request

// Output of a recurrent head group: out = RMS norm over each head's vdim values * w * sigmoid(g).
typedef struct nfk_head_norm_gate_params {
  const float* o;            // [T, ld_o]
  long long ld_o;
  const void* g;             // [T, ld_g]
  long long ld_g;
  const float* w;            // [heads * vdim_p]
  void* out;                 // [T, ld_out]
  long long ld_out;
  int T, heads, vdim, vdim_p;   // vdim_p: columns per head (padded)
  float eps;
  int dtype;
} nfk_head_norm_gate_params;
int nfk_head_norm_gate(const nfk_head_norm_gate_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Grouped-query attention with options (gqa.cu)
// ------------------------------------------------------------------------------------------------
// Pool of one layer as for nfk_attn_*: [pages][2 (K, V)][kv_heads][page_size][hd]; hd is the padded size of a head's
// keys and values (padding columns are zero).
// Per token: RMS norm of the whole query row and of the whole key row (all heads at once), keys and values to their
// page slot. v_mode 1 also keeps the values in v_first; 2 mixes them, v <- (1 - lambda) v + lambda v_first.
// rot: neighbouring columns 2i, 2i + 1 (i < rot_pairs) of every query and key head turn by the token's angles, table
// [T][rot_ld][2] of (cos, sin) as nfk_rope_table makes it; v_rot the same for the values.
typedef struct nfk_gqa_append_params {
  const void* src;           // [T, ld_src]: q at q_off, k at k_off, v at v_off, head h at column h * hd
  long long ld_src;
  int q_off, k_off, v_off;
  void* q_out;               // [T, heads * hd], null: queries are left where they are (no norm, no rotation)
  const float* q_w;          // [heads * hd] norm weights, null: no norm
  const float* k_w;          // [kv_heads * hd]
  void* v_first;             // [T, kv_heads * hd]
  int v_mode;
  float v_lambda;
  void* pool;
  const int* positions;
  const int* token_req;
  const int* kv_indptr;
  const int* kv_indices;
  const int* kv_first;
  int T, heads, kv_heads, hd, dim;    // dim: real size of a head's query and key
  int page_size, num_pages;
  float eps;
  int dtype;
  unsigned int* status;
  const float* rot;          // null: none
  const float* v_rot;
  int rot_pairs, rot_ld, v_pairs, v_ld;
} nfk_gqa_append_params;
int nfk_gqa_append(const nfk_gqa_append_params* p, cudaStream_t stream);

// Attention of the tokens [token_begin, token_begin + n_tokens), any sizes, bf16 or fp32: one CTA per token and head.
typedef struct nfk_gqa_attn_params {
  const void* q;             // [T, heads * hd]
  const void* pool;
  void* out;                 // [T, heads * hd]
  const int* positions;
  const int* token_req;
  const int* kv_indptr;
  const int* kv_indices;
  const int* kv_first;
  const float* sinks;        // [heads], null: none
  int token_begin, n_tokens, heads, kv_heads, hd, page_size, num_pages, window;
  float scale, softcap;      // softcap 0: none
  int dtype;
  unsigned int* status;
  const float* dist;         // as in nfk_attn_params
  int chunk;
  int ld_q;                  // elements from token to token of q; 0 = heads * hd
} nfk_gqa_attn_params;
int nfk_gqa_attn(const nfk_gqa_attn_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Attention with mixed heads (talk.cu)
// ------------------------------------------------------------------------------------------------
// Softmax weights w_g(i, j) of every head (window and sink as for nfk_gqa_attn), then
// out_h(i) = sum_j (sum_g talk[h][g] w_g(i, j)) v(j) with the values of h's own key/value head. v_rot: the output's
// neighbouring columns turn back by the token's angles (table [T][v_ld][2] of (cos, sin), v_pairs pairs per head).
// Pool as for nfk_gqa_append.
typedef struct nfk_talk_attn_params {
  const void* q;             // [T, heads * hd]
  const void* pool;
  void* out;                 // [T, heads * hd]
  const int* positions;
  const int* token_req;
  const int* kv_indptr;
  const int* kv_indices;
  const int* kv_first;
  const float* sinks;        // [heads], null: none
  const float* talk;         // [heads][heads]
  const float* v_rot;        // null: none
  int v_pairs, v_ld;
  int token_begin, n_tokens;
  int heads, kv_heads, hd, page_size, num_pages, window;   // window 0: none
  float scale;
  int dtype;
  unsigned int* status;
  int max_keys;              // decode: most keys that a token sees
  const int* items;          // prefill: [num_items][3] (request, first token, tokens: at most 16)
  int num_items;
} nfk_talk_attn_params;
// Tokens [token_begin, token_begin + n_tokens), any sizes (shared memory for a few rows of all heads permitting), bf16 or
// fp32: one CTA per token.
int nfk_talk_attn(const nfk_talk_attn_params* p, cudaStream_t stream);
// bf16, hd 64 or 128, at most 64 heads, `talk` enters the products in bf16. Tokens [token_begin, token_begin + n_tokens), a
// cluster of CTAs each:
int nfk_talk_attn_decode(const nfk_talk_attn_params* p, cudaStream_t stream);
// ... and portions:
int nfk_talk_attn_prefill(const nfk_talk_attn_params* p, cudaStream_t stream);
// Which of the two take these sizes: 1 = prefill, 2 = decode (for max_keys keys), added up.
int nfk_talk_attn_fits(int heads, int kv_heads, int hd, int max_keys);

// ------------------------------------------------------------------------------------------------
// Short convolution over time (short_conv.cu)
// ------------------------------------------------------------------------------------------------
// Per channel: y_t = act(sum_j w[j] x_(t - taps + 1 + j) (+ bias)) (+ x_t if residual), zeros before the sequence's start.
// The last taps - 1 inputs of a request are kept in its state: half ref & 1 is read, the other one written.
enum { NFK_CONV_NONE = 0, NFK_CONV_SILU = 1 };
typedef struct nfk_short_conv_params {
  const void* x;             // [T, ld_x]
  long long ld_x;
  void* out;                 // [T, ld_out], not x
  long long ld_out;
  const float* w;            // [taps][cols]
  const float* bias;         // [cols], null: none
  void* state;               // [slots][2][max(1, taps - 1)][cols], stored as x
  const int* state_slot;     // [B] 2 * slot + half
  const int* positions;
  const int* token_req;
  const int* qo_indptr;
  int row_begin, T;          // rows row_begin .. T - 1 (whole requests)
  int cols, taps, act, residual, num_slots, dtype;
  unsigned int* status;
} nfk_short_conv_params;
int nfk_short_conv(const nfk_short_conv_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Real-gated linear recurrent unit (rglru.cu)
// ------------------------------------------------------------------------------------------------
// Per channel: log a = log_a sigmoid(r + r_b), S <- a S + sqrt(1 - a^2) sigmoid(i + i_b) u; out = S gelu_tanh(y).
// Channels come in blocks of `block`: the gates' pre-activations of a block are its r columns, then its i columns.
// A request whose first token of the launch is at position 0 starts from zero.
typedef struct nfk_rglru_params {
  const void* u;             // [T, ld_u]
  long long ld_u;
  const void* y;             // [T, ld_y]
  long long ld_y;
  const float* gates;        // [T, ld_g]
  long long ld_g;
  const float* r_b;          // [cols]
  const float* i_b;
  const float* log_a;
  float* S;                  // [slots][cols]
  void* out;                 // [T, ld_out]
  long long ld_out;
  const int* positions;
  const int* qo_indptr;
  const int* state_slot;     // [B] 2 * slot (+ half, not used here)
  int req_begin, req_count, cols, block, num_slots;
  int dtype;
  unsigned int* status;
} nfk_rglru_params;
int nfk_rglru_decode(const nfk_rglru_params* p, cudaStream_t stream);    // one token per request
int nfk_rglru_prefill(const nfk_rglru_params* p, cudaStream_t stream);   // any number of tokens per request

// ------------------------------------------------------------------------------------------------
// Delta-rule recurrence (delta.cu)
// ------------------------------------------------------------------------------------------------
// Per head, q and k of head h being those of q/k head h / (heads / kv_heads) as unit vectors (x / sqrt(sum x^2 + unit_eps)),
// q times q_scale, with w = exp(-rate softplus(x + dt_bias)) per key channel and beta = sigmoid(b):
//   S <- diag(w) S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q
//   y = RMS norm of o (over the head's vdim_real values) * norm * sigmoid(g)
// A request whose first token of the launch is at position 0 starts from a zero state.
typedef struct nfk_delta_params {
  const void* qkv;           // [T, ld]: q at q_off + head * dim, k at k_off, v at v_off + head * vdim
  long long ld;
  int q_off, k_off, v_off;
  const float* x;            // [T, ld_x], head h at column h * dim
  long long ld_x;
  const float* beta;         // [T, ld_b], head h at column h
  long long ld_b;
  const void* g;             // [T, ld_g], head h at column h * vdim
  long long ld_g;
  const float* rate;         // [heads]
  const float* dt_bias;      // [heads * dim]
  const float* norm;         // [vdim]
  float* S;                  // [slots][heads][dim][vdim]
  void* y;                   // [T, ld_y]
  long long ld_y;
  const int* positions;
  const int* qo_indptr;
  const int* state_slot;     // [B] 2 * slot (+ half, not used here)
  int req_begin, req_count;  // decode: requests with one token each
  int heads, kv_heads, dim, vdim, vdim_real, num_slots;    // dim, vdim: padded to multiples of 8 (padding columns are zero)
  float q_scale, unit_eps, eps;
  int dtype;
  // prefill. o: fp32 [T, heads * vdim] of scratch rows. Token by token: seq_reqs [num_seq] requests. In chunks of 64 tokens
  // (bf16, dim and vdim up to 128): items [num_items][4] (request, first token, tokens, chunk of the request's portion), a
  // request's chunks one after the other, of num_portions requests (0: not said), and scratch: num_items * heads *
  // nfk_delta_item_floats(dim, vdim) floats.
  const int* seq_reqs;
  int num_seq;
  float* o;
  const int* items;
  int num_items;
  float* scratch;
  long long scratch_floats;
  unsigned int* status;
  int num_portions;          // requests whose chunks are listed; 0: not said
} nfk_delta_params;
long long nfk_delta_item_floats(int dim, int vdim);
int nfk_delta_decode(const nfk_delta_params* p, cudaStream_t stream);
int nfk_delta_prefill(const nfk_delta_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Mixture of experts (moe.cu)
// ------------------------------------------------------------------------------------------------
enum { NFK_SCORE_SIGMOID = 0, NFK_SCORE_SOFTMAX = 1, NFK_SCORE_SOFTMAX_ALL = 2 };
// NFK_SCORE_SOFTMAX_ALL: scores s = softmax(logits) over all outputs, choice scores s + correction, weights s times scale (not
// normed). `identity`: so many outputs behind the experts stand for the input itself: they take part in scores, groups and
// choice, but get no row; the sum of a token's weights of such choices goes to gate. group_max: a group counts by its
// largest choice score instead of the sum of the two largest.
// NFK_SCORE_SOFTMAX: the experts are chosen by logits + correction and weighted by the softmax of those sums over the
// chosen ones, times scale (groups as below). NFK_SCORE_SIGMOID:
// Scores s = sigmoid(logits); choice scores s + correction. Experts form `groups` equal runs of neighbours (1: no
// grouping); a group counts by the sum of its two largest choice scores and only experts of the best `keep` groups
// can be chosen. Weights: s of the `top` chosen ones over their sum, times scale. Ties go to the lower index.
// Every chosen expert's counter is increased; what it was before is the token's rank among the expert's rows.
typedef struct nfk_moe_route_params {
  const float* logits;       // [T, ld]: experts at columns 0 .., the shared expert's gate at gate_col (< 0: none)
  long long ld;
  const float* correction;   // [experts], null: none
  int* expert;               // [T][top]
  float* weight;             // [T][top]
  int* rank;                 // [T][top]
  int* counts;               // [experts], zero before the launch
  float* gate;               // [T] sigmoid of the gate column
  int T, experts, top, groups, keep, gate_col;
  float scale;
  int score;                 // NFK_SCORE_*
  int identity, group_max;   // identity > 0: no gate column
} nfk_moe_route_params;
int nfk_moe_route(const nfk_moe_route_params* p, cudaStream_t stream);

// Rows of h in expert order: row rank + (rows of the experts before) of out for every chosen expert of a token. Choices past the
// experts get no row and slot -1.
typedef struct nfk_moe_permute_params {
  const void* h;             // [T, ld_h]
  long long ld_h;
  void* out;                 // [>= T * top, ld_out]
  long long ld_out;
  const int* expert;
  const int* rank;
  const int* counts;
  int* slot;                 // [T][top]
  int T, top, experts, cols; // cols: a multiple of 8
  int dtype;
} nfk_moe_permute_params;
int nfk_moe_permute(const nfk_moe_permute_params* p, cudaStream_t stream);

// One product per expert over its rows of A (rows in expert order, counts per expert on the device):
// D = A B_e^T with lin_act, or with B2 the gated epilogue of nfk_gemm_bf16. Matrices of the experts are stacked: B [experts * N, ldb].
typedef struct nfk_moe_gemm_params {
  const void* A;             // [rows, lda]
  const void* B;
  const void* B2;            // up matrices, null: linear
  void* D;                   // [rows, ldd]
  const int* counts;
  long long lda, ldb, ldd;
  int rows;                  // most rows (T * top)
  int experts, N, K;         // N, K: multiples of 8
  int act;
  float act_limit, act_alpha, act_shift;
  int dtype, num_ctas;
  unsigned int* status;
  int lin_act;               // NFK_LIN_*
} nfk_moe_gemm_params;
int nfk_moe_gemm(const nfk_moe_gemm_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// WKV recurrence (wkv.cu)
// ------------------------------------------------------------------------------------------------
// out[t, s * ld_h + c] = h + (h' - h) mu[s][c] with h' the previous token's row: of the same request in this launch,
// of the state (half ref & 1 is read, the other one receives the request's last row), or zero at position 0.
typedef struct nfk_token_shift_params {
  const void* h;             // [T, ld_h]
  long long ld_h;
  void* out;                 // [T, n_mix * ld_h]
  const float* mu;           // [n_mix][ld_h]
  void* state;               // [slots][2][ld_h]
  const int* state_slot;     // [B] 2 * slot + half
  const int* positions;
  const int* token_req;
  const int* qo_indptr;
  int T, n_mix, num_slots;
  int dtype;
  unsigned int* status;
} nfk_token_shift_params;
int nfk_token_shift(const nfk_token_shift_params* p, cudaStream_t stream);

// Per head, with w_t = exp(-exp(x_t)) per key channel:
//   o_t = (S + diag(u) k_t v_t^T)^T r_t;  S <- diag(w_t) S + k_t v_t^T
//   y_t = RMS norm of o_t (over the head's `dim_real` values) * norm * silu(g_t)
// A request whose first token of the launch is at position 0 starts from a zero state.
typedef struct nfk_wkv_params {
  const void* rkvg;          // [T, ld]: r, k, v, g at their offsets, head h at column h * dim
  long long ld;
  int r_off, k_off, v_off, g_off;
  const float* x;            // [T, ld_x] logarithm of the decay's negative logarithm
  long long ld_x;
  const float* u;            // [heads * dim]
  const float* norm;         // [heads * dim]
  float* S;                  // [slots][heads][dim][dim], key channel first
  void* y;                   // [T, ld_y]
  long long ld_y;
  const int* positions;
  const int* qo_indptr;
  const int* state_slot;     // [B] 2 * slot (+ half, not used here)
  int req_begin, req_count;  // decode: requests with one token each
  int heads, dim, dim_real, num_slots;
  float eps;
  int dtype;
  // prefill. Token by token: seq_reqs [num_seq] requests, o: fp32 [T, heads * dim] of scratch rows. In chunks of 64 tokens
  // (bf16): items [num_items][4] (request, first token, tokens, chunk of the request's portion), a request's chunks one
  // after the other, and scratch: num_items * heads * (dim * dim + dim) floats.
  const int* seq_reqs;
  int num_seq;
  float* o;
  const int* items;
  int num_items;
  float* scratch;
  long long scratch_floats;
  unsigned int* status;
} nfk_wkv_params;
int nfk_wkv_decode(const nfk_wkv_params* p, cudaStream_t stream);
int nfk_wkv_prefill(const nfk_wkv_params* p, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// KV offload (kv_offload.cu): gather / scatter whole pages between the pool and a staging buffer
// ------------------------------------------------------------------------------------------------
// page_bytes = 2*kv_heads*page_size*head_dim*2. direction 0: staging[i] = pool[page_ids[i]];
// direction 1: pool[page_ids[i]] = staging[i].
int nfk_kv_move_pages(void* pool, void* staging, const int* page_ids, int n_pages,
                      long long page_bytes, int num_pages, int direction, int num_ctas,
                      unsigned int* status, cudaStream_t stream);

// ------------------------------------------------------------------------------------------------
// Tensor-parallel collectives on a symmetric heap (collectives.cu)
// ------------------------------------------------------------------------------------------------
typedef struct nfk_comm_ctx {
  void* heap[8];       // base of every rank's symmetric heap as mapped into this process
  int rank, nranks;
} nfk_comm_ctx;

typedef struct nfk_allreduce_params {
  nfk_comm_ctx ctx;
  long long buf_off;      // byte offset of the bf16 [rows, ld] buffer inside the heap (summed in place)
  long long flag_off;     // byte offset of this op's 128-byte flag block
  int rows, cols;
  long long ld;           // elements
  int epoch;              // monotonic per call on this flag block (e.g. iteration number)
  int num_ctas;
  const void* norm_w;     // optional: RMSNorm weight [cols]; normed rows go to norm_out on all ranks
  long long norm_out_off; // byte offset of the bf16 [rows, norm_ld] output inside the heap
  long long norm_ld;
  float eps;
  unsigned int* status;
  int push_sum;           // 1: write the sum back into the buffer on every rank (in-place all-reduce)
  const void* resid;      // optional local bf16 [rows, resid_ld]: owned rows are added to the sum
  long long resid_ld;
  void* sum_out;          // optional local bf16 [rows, sum_ld]: owned rows of the sum are stored here
  long long sum_ld;
  int src_mode;           // 0: pull row i from every rank's buffer. 1: the partials were pushed here by a
                          //    NFK_EPI_REDUCE_SCATTER GEMM: owned row k of rank r's partial sits in the local
                          //    slab at buf_off + (r * slab_rows + k) * ld (no NVLink loads, no ready signal)
                          //    2: rank r's buffer holds columns [r*cols/nranks, (r+1)*cols/nranks) of every row (the
                          //    output of an N-split GEMM): an owned row is gathered from the ranks' column blocks
                          //    instead of summed, then residual / norm / pushes as in mode 0
  int slab_rows;
  int wide;               // 1 (8 ranks): twice the loads in flight per phase, the norm pass re-reads the stored sum
  // Optional row-block flags for a consumer that starts before this collective has finished (see
  // nfk_gemm_params::gate_flags): gate_off is the heap offset of [ceil(rows/128)][8] words (same offset on
  // every rank), gate_cnt a local array of ceil(rows/128) zero-initialised words (this rank's rows done per
  // block; reset by the kernel). Once a rank has pushed all the normed rows it owns inside block b it writes
  // `epoch` into word [b][rank] on every rank. Needs norm_w / norm_out (the pushed rows are what is gated).
  long long gate_off;
  unsigned int* gate_cnt;
  // 1: the normed rows this rank owns are stored into its OWN copy of norm_out only and the kernel ends
  // without the exit handshake: the caller delivers them to the peers with copy-engine copies (no SM
  // involved, see parallel/collectives.py) and closes with nfk_comm_barrier. Needs norm_w; no gate flags.
  int push_mode;
  void* mc_heap;          // optional: the heaps' NVLink multicast mapping (one address that stands for the same
                          //    offset on every rank). Non-null selects the in-switch form: owned rows are summed by
                          //    multimem.ld_reduce and results are written to all ranks by multimem.st (src_mode 0 only)
} nfk_allreduce_params;
int nfk_allreduce(const nfk_allreduce_params* p, cudaStream_t stream);

typedef struct nfk_allgather_params {
  nfk_comm_ctx ctx;
  long long buf_off;       // symmetric buffer holding nranks shards, shard r at buf_off + r*shard_stride
  long long shard_bytes, shard_stride, flag_off;
  int epoch, num_ctas, handshake_in;
  unsigned int* status;
  // Column-wise form (rows > 1): the buffer is [rows][...] with row_stride bytes between rows, and
  // rank r owns the shard_bytes starting at byte r*shard_stride of every row (its column block).
  // rows <= 1 is the flat form above.
  int rows;
  long long row_stride;
} nfk_allgather_params;
int nfk_allgather(const nfk_allgather_params* p, cudaStream_t stream);

typedef struct nfk_comm_barrier_params {
  nfk_comm_ctx ctx;
  long long flag_off;
  int epoch;
  unsigned int* status;
} nfk_comm_barrier_params;
int nfk_comm_barrier(const nfk_comm_barrier_params* p, cudaStream_t stream);

// Symmetric heap plumbing: allocate (zero-filled), export / open CUDA IPC handles (64 bytes).
int nfk_symm_alloc(void** out, long long bytes);
int nfk_symm_free(void* p);
int nfk_ipc_get_handle(void* ptr, unsigned char* out64);
int nfk_ipc_open_handle(const unsigned char* in64, void** out);
int nfk_ipc_close_handle(void* p);

// ------------------------------------------------------------------------------------------------
// Uniform launch ABI (abi.cu): every op is also reachable as  int fn(const <params>*, cudaStream_t)
// so that a generic executor can replay a list of (function pointer, parameter block) pairs.
// ------------------------------------------------------------------------------------------------
typedef struct nfk_norm_params {
  void* out; const void* x; const void* w; void* resid;   // resid != NULL: resid += x, out = norm(resid)
  int rows, cols; float eps;
} nfk_norm_params;
typedef struct nfk_embedding_params {
  void* out; const void* table; const int* host_ids; const int* feedback_src; const int* prev_tokens;
  int* ids_out; int n_tokens, hidden, vocab; unsigned int* status;
} nfk_embedding_params;
typedef struct nfk_gather_params {
  void* out; const void* in; const int* rows_idx; int n, cols; long long ld_in; int in_rows;
  unsigned int* status;
} nfk_gather_params;
typedef struct nfk_argmax_params {
  int* idx_out; float* val_out; const void* logits; int rows, cols; long long ld; int col_offset;
  int dtype;   // NFK_BF16 / NFK_F32
} nfk_argmax_params;
typedef struct nfk_argmax_combine_params {
  int* idx_out; const float* cand_val; const int* cand_idx; int shards, rows;
} nfk_argmax_combine_params;
typedef struct nfk_copy_cols_params {
  void* out; long long ld_out; const void* in; long long ld_in; int rows, cols;
} nfk_copy_cols_params;
typedef struct nfk_memcpy_params {   // plain async copy (any direction); elem_bytes * count bytes
  void* dst; const void* src; long long elem_bytes; int count;
} nfk_memcpy_params;
typedef struct nfk_memcpy2d_params {  // strided async copy: `height` rows of `width` bytes, row pitches in bytes
  void* dst; const void* src; long long dpitch, spitch, width; int height;
} nfk_memcpy2d_params;
typedef struct nfk_kv_move_params {
  void* pool; void* staging; const int* page_ids; int n_pages; long long page_bytes; int num_pages;
  int direction; int num_ctas; unsigned int* status;
} nfk_kv_move_params;

int nfk_norm_p(const nfk_norm_params* p, cudaStream_t s);
int nfk_embedding_p(const nfk_embedding_params* p, cudaStream_t s);
int nfk_gather_p(const nfk_gather_params* p, cudaStream_t s);
int nfk_argmax_p(const nfk_argmax_params* p, cudaStream_t s);
int nfk_argmax_combine_p(const nfk_argmax_combine_params* p, cudaStream_t s);
int nfk_copy_cols_p(const nfk_copy_cols_params* p, cudaStream_t s);
int nfk_memcpy_p(const nfk_memcpy_params* p, cudaStream_t s);
typedef struct nfk_sleep_params { int micros; } nfk_sleep_params;   // nfk_sleep as an op of the graph
int nfk_sleep_p(const nfk_sleep_params* p, cudaStream_t s);
int nfk_kv_move_p(const nfk_kv_move_params* p, cudaStream_t s);

#ifdef __cplusplus
}
#endif
