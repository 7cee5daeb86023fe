/*
 * llmb200_kernels.h -- thin C ABI over the sm_100a kernels of the decode path.
 *
 * Plain pointers and sizes only. Every pointer named d_* is CUDA device memory
 * on the current device; `stream` is a cudaStream_t passed as void*. Functions
 * return 0 on success, a positive cudaError_t value when CUDA reports one and
 * a negative B200_E_* code for rejected arguments. Nothing here allocates
 * device memory.
 *
 * Each launcher states which reference dispatch(es) it stands in for
 * (src/nn/fast_metal.m line of the metal_enqueue_* function, and the kernel in
 * shaders/q8_kernels.metal).
 *
 * Packed weight layout ("row-sliced"):
 *   Q8_0  row r = cols int8 quants, then cols/32 binary16 scales; rows are
 *         row_stride bytes apart, row_stride = round_up(34*cols/32, 16).
 *   F16   row r = cols binary16 values; row_stride = round_up(2*cols, 16).
 *   BF16  row r = cols bfloat16 values; row_stride = round_up(2*cols, 16).
 *   F32   row r = cols fp32 values;     row_stride = round_up(4*cols, 16).
 * Values are exactly those of the reference's 34-byte block stream / half
 * array; only the placement differs, so that every 16-byte load of a row is
 * aligned and a warp reads 512 contiguous bytes.
 */
#ifndef LLMB200_KERNELS_H
#define LLMB200_KERNELS_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define B200_E_BADARG   (-1)
#define B200_E_TOOLARGE (-2)
#define B200_E_STATE    (-3)

#define B200_WT_Q8   0
#define B200_WT_F16  1
#define B200_WT_BF16 2
#define B200_WT_F32  3

#define B200_MAX_PEERS 8

/* Bytes between consecutive rows of a packed matrix with `cols` columns. */
size_t b200_packed_row_stride(int wtype, int cols);

/* fp32 [rows, cols] (leading dimension ld floats, device) -> packed Q8_0 rows.
 * Source row r lands in packed row dst_row0 + r*dst_row_step.
 * Replaces quantize_row_q8/wmat_create_q8 (src/nn/wmat.c:19-61); bit-exact. */
int b200_q8_pack(const float *d_src, long long ld, int rows, int cols,
                 void *d_dst, long long dst_row_stride, int dst_row0, int dst_row_step,
                 void *stream);
/* fp32 rows -> bfloat16 (round to nearest even) or fp32 packed rows (wtype B200_WT_BF16 / B200_WT_F32). Any
 * column count; the bytes of a row from cols up to dst_row_stride are written as zeros, so that a matrix
 * can be given padding columns. No counterpart in the reference. */
int b200_cast_pack(int wtype, const float *d_src, long long ld, int rows, int cols,
                   void *d_dst, long long dst_row_stride, int dst_row0, int dst_row_step, void *stream);
/* Same for F16 (src/nn/wmat.c:63-75). */
int b200_f16_pack(const float *d_src, long long ld, int rows, int cols,
                  void *d_dst, long long dst_row_stride, int dst_row0, int dst_row_step,
                  void *stream);
/* Packed Q8_0 rows -> the reference's canonical stream of 34-byte blocks
 * {u16 d; i8 qs[32]} (src/nn/wmat.c:14-17), rows*cols/32 blocks, row-major. */
int b200_q8_unpack_blocks(const void *d_packed, long long row_stride, int rows, int cols,
                          void *d_blocks, void *stream);

/* ------------------------------------------------------------------------
 * Fused matrix-vector product  y = W . f(x)
 *
 * One launch covers what the reference enqueues as rms_norm + q8_matvec /
 * f16_matvec (+ residual_add, silu_mul / gelu_mul, CPU embedding copy, CPU
 * argmax): src/nn/fast_metal.m:253-289, 309-341, 428-462 and
 * src/nn/fast_inference.c:386-392, 469-476.
 *
 * Input assembly (in_mode), all in fp32:
 *   B200_IN_VEC    x = in_vec[cols]
 *   B200_IN_RESID  h = resid_in + S, S = sum over n_slots of slots[s][0..cols)
 *                  (if slot_norm_gamma: S <- rmsnorm(S) * slot_norm_gamma first);
 *                  block 0 stores h to resid_out; x = h
 *   B200_IN_EMBED  h = emb[tokens[*pos]][0..cols) * emb_scale; stored to
 *                  resid_out by block 0; x = h. BF16 / F32 weights: emb_pos[*pos][0..cols) is added when given
 *                  (rows past emb_pos_rows read the last one), then slot_norm_gamma / slot_norm_beta
 *                  make h its layer norm, and x = *mix_coef * h when mix_coef is given
 *   B200_IN_POSTNORM (BF16 / F32 weights) h = norm(in_vec) * slot_norm_gamma; block 0 stores h to
 *                  post_copy (if not NULL); x = mix_in ? mix_in + *mix_coef * h : h, stored to
 *                  resid_out by block 0 (if not NULL)
 * then, if norm_gamma != NULL, x <- x * rsqrt(mean(x^2)+eps) * norm_gamma. With norm_groups > 1 the
 * norms of BF16 / F32 launches treat that many equal consecutive parts of the vector separately;
 * norm_dim (0 = cols) is the length they run over when the columns past it are padding. A norm that is
 * given a bias (norm_beta, slot_norm_beta; BF16 / F32) is a layer norm: (x - mean) / sqrt(variance + eps)
 * * gamma + beta.
 *
 * Output (out_mode):
 *   B200_OUT_STORE  out[p][out_offset + r] = y[r] for every peer p < n_out
 *   B200_OUT_GLU    rows come in (gate, up) pairs: out[0][out_offset + r/2] =
 *                   act(y[r]) * y[r+1], act = SiLU (0) or tanh-GELU (1). glu_rows > 0: only rows below
 *                   it are pairs, row r above goes to out2[r - glu_rows] as it is
 *   B200_OUT_GATED  (BF16 / F32 weights) out[0][r] = resid_alpha * out_resid[r]
 *                   + sigmoid(out_gate[r] + out_gate_bias[r]) * y[r]
 *   B200_OUT_STREAMS (BF16 / F32 weights) the result joins n_streams residual streams X_s: X'_t[r] =
 *                   sum over s of mix[s][t] * X_s[r] + spread[t] * y[r], stored at streams_out +
 *                   t * streams_out_stride, and out[0][r] = sum over t of take[t] * X'_t[r], what the next
 *                   reader sees. connect = mix (from, to) | spread | take, n_streams * (n_streams + 2) floats.
 *                   streams_in_stride 0: all old streams are one vector
 * B200_OUT_STORE with act = B200_ACT_RELU2 (BF16 / F32) stores max(y, 0)^2.
 * Layer norms, learned positions, streams and the squared relu form one family of kernels, post-norm inputs,
 * GLU, gated outputs, depth sums, RMS norms and the cap another: a BF16 / F32 launch uses one of the two.
 * BF16 / F32 launches can also cap what they store, y <- softcap * tanh(y / softcap), and form a depth
 * sum for the rows they own, hist_out[r] = sum over j < hist_n of hist_coef[j] * hist[j * hist_stride + r].
 * With d_argmax_scratch != NULL (B200_OUT_STORE only) the launch also leaves
 * the largest y[r] and its row index plus out_offset (first one on ties, as
 * the reference's argmax) in *d_argmax_val[p] / *d_argmax_idx[p], p < n_argmax_out.
 *
 * Tensor-parallel hand-shake (all optional, n_wait = 0 / n_signal = 0 to
 * disable): before reading `slots` the kernel waits, with an iteration limit,
 * until wait_flags[i] >= E for i < n_wait, E = *epoch * epoch_mul + epoch_add;
 * after its last store it writes E into signal_flags[p][signal_index], p < n_signal. A wait
 * that runs out sets *err = 1 and the kernel carries on without hanging.
 * ---------------------------------------------------------------------- */
enum { B200_IN_VEC = 0, B200_IN_RESID = 1, B200_IN_EMBED = 2, B200_IN_POSTNORM = 3 };
enum { B200_OUT_STORE = 0, B200_OUT_GLU = 1, B200_OUT_GATED = 2, B200_OUT_STREAMS = 3 };
enum { B200_ACT_SILU = 0, B200_ACT_GELU_TANH = 1, B200_ACT_RELU2 = 2 };
#define B200_MAX_STREAMS 8

typedef struct b200_matvec_args {
    /* weights */
    const void *d_w; long long row_stride; int rows, cols, wtype;
    /* input assembly */
    int in_mode;
    const float *d_in_vec;
    const float *d_resid_in; float *d_resid_out;
    const float *d_slots; int n_slots; long long slot_stride;   /* floats between slots */
    const float *d_slot_norm_gamma;
    const float *d_emb; const int *d_tokens; const int *d_pos; float emb_scale;
    int emb_rows;                  /* rows of d_emb; an id outside [0, emb_rows) is read as id 0 */
    const float *d_norm_gamma; float eps;
    /* output */
    int out_mode, act;
    float *d_out[B200_MAX_PEERS]; int n_out; long long out_offset;
    float *d_argmax_scratch;                       /* 2 words per block, or NULL: no argmax */
    float *d_argmax_val[B200_MAX_PEERS];           /* [0] of each receives the largest y */
    int   *d_argmax_idx[B200_MAX_PEERS];           /* [0] of each receives its row + out_offset */
    int    n_argmax_out;
    /* bookkeeping done by the last block to finish */
    unsigned *d_ticket;            /* one zero-initialised word; required when any of the below is used */
    int advance_pos;               /* (*d_pos_rw)++ */
    int *d_pos_rw;
    int advance_epoch;             /* *d_epoch_rw = *d_epoch + 1 */
    unsigned *d_epoch_rw;
    int *d_next_token; const int *d_prompt_len;   /* tokens[pos+1] = argmax unless pos+1 < *prompt_len */
    /* tensor-parallel flags */
    const unsigned *d_wait_flags; int n_wait;
    unsigned *d_signal_flags[B200_MAX_PEERS]; int n_signal, signal_index;
    const unsigned *d_epoch; int epoch_mul, epoch_add;   /* flag value = *d_epoch * epoch_mul + epoch_add */
    int *d_err;
    /* launch shape: 0 = choose (a multiple of the SM count) */
    int grid;
    int use_pdl;                   /* programmatic dependent launch: prefetch weights under the previous kernel's tail */
    /* optional: block 0 also stores the assembled (summed, normalised) input vector here, cols floats --
     * what a LoRA side path multiplies by A (src/nn/fast_inference.c:406-421 reads mb_ln_out) */
    float *d_in_copy;
    /* iterations of the bounded wait on d_wait_flags before the kernel gives up and sets *d_err = 1
     * (0 = default, about a second) */
    int spin_limit;
    /* BF16 / F32 weights only (see above); all zero otherwise */
    int norm_dim, norm_groups;
    float *d_post_copy; const float *d_mix_in; const float *d_mix_coef;
    const float *d_out_resid, *d_out_gate, *d_out_gate_bias; float resid_alpha;
    const float *d_hist; int hist_n; long long hist_stride; const float *d_hist_coef; float *d_hist_out;
    int glu_rows; float *d_out2;
    float softcap;                 /* 0 = none */
    const float *d_norm_beta, *d_slot_norm_beta;
    const float *d_emb_pos; int emb_pos_rows;
    const float *d_streams_in; long long streams_in_stride;
    float *d_streams_out; long long streams_out_stride;
    const float *d_connect; int n_streams;
} b200_matvec_args;

int b200_matvec(const b200_matvec_args *a, void *stream);

/* ------------------------------------------------------------------------
 * Decode attention for one new token over an F16 KV cache, split over the
 * sequence. One launch covers per_head_rms_norm(q), per_head_rms_norm(k),
 * rope, kv_cache_store and attention of the reference
 * (src/nn/fast_metal.m:343-426; shaders/q8_kernels.metal:165-331).
 *
 *   qkv        fp32 [n_q*hd | n_kv*hd | n_kv*hd] of the new token (unnormalised)
 *   q/k_gamma  [hd] or NULL (no QK-norm)
 *   inv_freq   [hd/2] fp32, 1/theta^(2d/hd); angle = pos * inv_freq[d]
 *   k/v_cache  binary16 [n_kv][max_seq][hd]; row *pos is written by this launch
 *   out        fp32 [n_q*hd]
 *   scratch    fp32, b200_attn_scratch_floats(n_q, hd, n_split) floats
 *   tickets    n_kv zero-initialised words
 * Keys 0..*pos are attended (no window), scores scaled by 1/sqrt(hd). A position outside
 * [0, max_seq) is ignored: nothing is written or read, the output keeps its contents.
 * ---------------------------------------------------------------------- */
typedef struct b200_attn_args {
    const float *d_qkv; const float *d_q_gamma; const float *d_k_gamma; const float *d_inv_freq;
    void *d_k_cache; void *d_v_cache;
    float *d_out; float *d_scratch; unsigned *d_tickets;
    const int *d_pos;
    int n_q, n_kv, hd, max_seq, n_split;
    float eps;
    int use_pdl;
    /* Batched form (several sequences at the same position, one launch): n_items > 1 adds a grid
     * dimension; item i reads d_qkv + i*qkv_item_stride, its own caches at + i*cache_item_stride halves,
     * writes d_out + i*out_item_stride and uses scratch / tickets slice i (b200_attn_scratch_floats and
     * n_kv words per item). 0 or 1 = one sequence. */
    int n_items;
    long long qkv_item_stride, cache_item_stride, out_item_stride;
} b200_attn_args;

size_t b200_attn_scratch_floats(int n_q, int hd, int n_split);
int    b200_attn_decode(const b200_attn_args *a, void *stream);

/* No counterpart in the reference. b200_attn_decode for callers that cannot allocate device memory --
 * a process whose GPU memory was carved up completely at start-up, or a loop that must not risk the
 * device-wide synchronisation a cudaMalloc can cause. a->d_scratch and a->d_tickets are ignored; the
 * partial results go to arrays built into the library (held by every GPU that loads it until the
 * process exits). Limits: n_q * n_split * (hd + 2) <= B200_ATTN_STATIC_SCRATCH_FLOATS and
 * n_kv <= B200_ATTN_STATIC_MAX_KV_HEADS, one sequence per call (n_items <= 1: the batched form indexes
 * scratch and tickets by item); anything larger is refused with B200_E_TOOLARGE and a message on stderr. Calls no cudaMalloc/cudaFree. The first call on a device looks up the arrays'
 * device addresses and should therefore come before any stream capture. All calls share the arrays:
 * two calls whose kernels may overlap on the GPU (different streams) race with each other. */
#define B200_ATTN_STATIC_SCRATCH_FLOATS (1 << 18)      /* 1 MiB */
#define B200_ATTN_STATIC_MAX_KV_HEADS   64
int b200_attn_decode_static(const b200_attn_args *a, void *stream);

/* ------------------------------------------------------------------------
 * Latent attention: keys and values of all heads are linear maps of one low-rank vector per token, and
 * one rotated key part is shared by the heads, so the cache holds kv_rank + rot_dim numbers a token.
 *
 *   q     head by head [dim unrotated | rot_dim rotated]
 *   c     = rms_norm(dkv[0 .. kv_rank)) * dkv_gamma
 *   kr    = rotate(dkv[kv_rank .. kv_rank + rot_dim))
 *   score = scale * (q_unrotated . (W_uk c) + rotate(q_rotated) . kr)   over the visible positions
 *   out   = sigmoid(gate) * sum softmax(score) (W_uv c)
 *
 * Rotation: the pair (2i, 2i+1), i < rot_dims/2, turns by the angle whose (cos, sin) d_rope holds,
 * [max_seq][rot_dims/2][2]; the rest of the rotated part passes unchanged. Position i sees j with
 * 0 <= i - j < window (window <= 0: every j <= i).
 *
 * With up8(n) = n rounded up to a multiple of 8: a cache row is [up8(kv_rank) | up8(rot_dim)] elements of
 * the type `wtype` names (BF16 or F32), padding zero. d_w_uk_t: per head [kv_rank][up8(dim)] (the
 * transposed map). d_w_kv: per head up8(dim) rows of W_uk and up8(vdim) rows of W_uv, up8(kv_rank)
 * columns. The decode form's vectors are fp32 but for d_qlat.
 *
 * Decode (b200_latent_decode, three launches): one new token at *d_pos. The query is moved into the latent
 * space (q_lat = W_uk^T q), the scores and the weighted sum run over cache rows with all heads sharing
 * the row loads, split over the sequence, and W_uv is applied once to the merged sum.
 * Rows (b200_latent_rows_*): n_rows tokens from position pos0 on. _prep writes their cache rows and
 * d_q_rows; the caller forms d_kv = cache rows x d_w_kv^T for positions kv_row0 .. pos0 + n_rows - 1;
 * _attend runs the attention (BF16: tensor cores, F32: CUDA cores).
 * ---------------------------------------------------------------------- */
typedef struct b200_latent_args {
    int wtype;
    int heads, dim, rot_dim, rot_dims, vdim, kv_rank, window, max_seq;
    float scale, eps;
    const float *d_q, *d_dkv, *d_gate;   /* one token, or n_rows rows proj_ld floats apart */
    const float *d_dkv_gamma, *d_rope;
    void *d_cache;
    const void *d_w_uk_t, *d_w_kv;
    /* decode */
    void *d_qlat;                        /* [heads][up8(kv_rank) + up8(rot_dim)] elements of the type `wtype` names */
    float *d_part;                       /* [heads][n_split][up8(kv_rank) + 8] */
    float *d_out;                        /* [heads * vdim] */
    const int *d_pos;
    int n_split, use_pdl;
    /* rows */
    int n_rows, pos0, kv_row0;
    long long proj_ld;
    void *d_q_rows;                      /* [n_rows][heads][up8(dim) + up8(rot_dim)] */
    const void *d_kv; long long kv_ld;   /* [pos0 + n_rows - kv_row0] rows of [heads][up8(dim) + up8(vdim)], kv_ld elements apart */
    void *d_out_rows; long long out_ld;  /* [n_rows] rows of heads * vdim, out_ld elements apart */
} b200_latent_args;

/* Splits of the sequence worth launching for this shape (1 .. 256). */
int b200_latent_splits(int heads, int window, int max_seq);
int b200_latent_decode(const b200_latent_args *a, void *stream);
int b200_latent_rows_prep(const b200_latent_args *a, void *stream);
int b200_latent_rows_attend(const b200_latent_args *a, void *stream);

/* ------------------------------------------------------------------------
 * Grouped-query attention with normed queries and keys, no rotation. Per position:
 *   q = rms_norm(q head) * q_gamma * q_scale[position], k = rms_norm(k head) * k_gamma   (gammas shared by heads)
 *   score = scale * (q . k), then softcap * tanh(score / softcap) when softcap > 0
 * softmax over every earlier position and its own; query head h reads key / value head h / (heads / kv_heads).
 * The caches hold [kv_heads][max_seq] rows of up8(dim) / up8(vdim) elements of the type `wtype` names (BF16 or
 * F32), padding zero.
 * Decode (b200_gqa_decode, one launch): the token at *d_pos; writes its cache rows. A position outside
 * [0, max_seq) is ignored. d_tickets: kv_heads * heads zero-initialised words, zero again afterwards.
 * Rows: n_rows tokens from position pos0 on. _prep writes their cache rows and d_q_rows, _attend runs the
 * attention (BF16: tensor cores, F32: CUDA cores).
 * ---------------------------------------------------------------------- */
typedef struct b200_gqa_args {
    int wtype;
    int heads, kv_heads, dim, vdim, max_seq;
    float scale, softcap, eps;
    const float *d_q, *d_k, *d_v;        /* one token, or n_rows rows proj_ld floats apart */
    const float *d_q_gamma, *d_k_gamma;  /* [dim] */
    const float *d_q_scale;              /* [max_seq] or NULL */
    void *d_k_cache, *d_v_cache;
    /* decode */
    float *d_part;                       /* [heads][n_split][up8(vdim) + 8] */
    unsigned *d_tickets;
    float *d_out;                        /* [heads * vdim] */
    const int *d_pos;
    int n_split, use_pdl;
    /* rows */
    int n_rows, pos0;
    long long proj_ld;
    void *d_q_rows;                      /* [n_rows][heads][up8(dim)] */
    void *d_out_rows; long long out_ld;  /* [n_rows] rows of heads * vdim, out_ld elements apart */
} b200_gqa_args;

/* Clusters of blocks that share the sequence for this shape (1 .. 64). */
int b200_gqa_splits(int wtype, int heads, int kv_heads, int dim, int vdim, int max_seq);
int b200_gqa_decode(const b200_gqa_args *a, void *stream);
int b200_gqa_rows_prep(const b200_gqa_args *a, void *stream);
int b200_gqa_rows_attend(const b200_gqa_args *a, void *stream);

/* ------------------------------------------------------------------------
 * Gated linear attention: per head a state S [dim][vdim] in fp32 that decays by a factor per key channel,
 *   a = logistic(W_a2 f + a2_bias)^(1/tau),  S <- diag(a) S + k v^T,  o = S^T (q * q_scale)
 * then o is RMS-normed over vdim (norm_gamma, shared by heads) and multiplied by silu(gate).
 * f (rank numbers) is the low-rank input of the decay; d_a2 is [heads * dim][up4(rank)] fp32, padding zero.
 * Everything from the projections on is fp32.
 *
 * States are kept per position: the state before position p is in slot p mod n_slots of d_state
 * [n_slots][heads][dim][up8(vdim)] (padding zero) and the one after it goes to the next slot, so running a position again gives the
 * same result, as with a key cache. Before position 0 the state is zero, whatever the slot holds.
 * Decode (b200_gla_decode, one launch): the token at *d_pos. Rows (b200_gla_rows): n_rows tokens from position
 * pos0 on, cut into chunks of 64: their scores in parallel, then the states chunk by chunk, then all outputs.
 * ---------------------------------------------------------------------- */
#define B200_GLA_CHUNK 64
typedef struct b200_gla_args {
    int wtype;                           /* element type of d_out_rows */
    int heads, dim, vdim, rank, n_slots;
    float tau, q_scale, eps;
    const float *d_q, *d_k, *d_v, *d_gate, *d_f;   /* one token, or n_rows rows proj_ld floats apart */
    const float *d_a2, *d_a2_bias, *d_norm_gamma;
    float *d_state;
    /* decode */
    float *d_out;                        /* [heads * vdim] */
    const int *d_pos;
    int use_pdl;
    /* rows; n_chunks = (n_rows + 63) / 64 */
    int n_rows, pos0;
    long long proj_ld;
    /* scratch: three bfloat16 planes (a value as a sum of three) where nothing else is said, 16-byte aligned */
    void *d_qd, *d_kd;                   /* [n_chunks][heads][3][64][up16(dim)]: queries and keys times their decays */
    void *d_values;                      /* [n_chunks][heads][3][64][up8(vdim)] */
    void *d_scores;                      /* [n_chunks][heads][3][64][64] */
    void *d_chunk_state;                 /* [n_chunks][heads][3][dim][up8(vdim)]: the state before each chunk */
    float *d_decay;                      /* fp32 [n_chunks][heads][up8(dim)]: log2 of the decay over a whole chunk */
    float *d_o;                          /* fp32 [n_rows][heads * vdim]; vdim > 128 only */
    void *d_out_rows; long long out_ld;  /* [n_rows] rows of heads * vdim, out_ld elements apart */
} b200_gla_args;
int b200_gla_decode(const b200_gla_args *a, void *stream);
int b200_gla_rows(const b200_gla_args *a, void *stream);

/* ------------------------------------------------------------------------
 * Row-wise steps of a prompt portion. Rows are ld floats apart; columns dim .. ld-1 are padding and are
 * written as zeros. out_h (BF16 copies for the tensor-core products) may be NULL.
 * ---------------------------------------------------------------------- */
/* x[m] = scale * emb[tokens[m]], emb [vocab][ld]. */
int b200_rows_embed(const float *emb, const uint32_t *tokens, int rows, int vocab, int ld, float scale,
                    float *x, void *out_h, void *stream);
/* z = alpha * x + sigmoid(gate + bias) * y; xn = grouped RMS norm of z times gamma, stored to `norm_out`;
 * with hist_n > 0: out = sum over j < hist_n of coef[j] * hist[j][m] + coef[hist_n] * xn, else out = xn.
 * hist[j] is [rows][ld], hist_stride floats apart. out may equal norm_out when hist_n == 0. */
typedef struct b200_rows_postnorm_args {
    const float *x, *y; long long y_ld;
    const float *gate; long long gate_ld; const float *gate_bias;
    const float *gamma;
    float alpha, eps;
    int rows, dim, ld, groups;
    float *norm_out;
    const float *hist; int hist_n; long long hist_stride; const float *coef;
    float *out; void *out_h;
} b200_rows_postnorm_args;
int b200_rows_postnorm(const b200_rows_postnorm_args *a, void *stream);
/* Residual streams, one sublayer's result y joined in: X'_t[m] = sum over s of mix[s][t] * X_s[m] + spread[t] * y[m]
 * (connect as in B200_OUT_STREAMS), X_s at streams_in + s * streams_in_stride, X'_t at streams_out + t *
 * streams_out_stride (NULL: not kept), u[m] = sum over t of take[t] * X'_t[m] (stored to u_out when given), and the
 * layer norm of u (gamma, beta) to out, element type wtype (out NULL: no norm). */
typedef struct b200_rows_streams_args {
    const float *streams_in; long long streams_in_stride;
    const float *y; long long y_ld;
    const float *connect; int n_streams;
    const float *gamma, *beta; float eps;
    int rows, dim, ld, wtype;
    float *streams_out; long long streams_out_stride;
    float *u_out;
    void *out;
} b200_rows_streams_args;
int b200_rows_streams(const b200_rows_streams_args *a, void *stream);
/* The rows that all streams start from, x[m] = layer_norm(emb[tokens[m]] + emb_pos[pos0 + m]) * emb_gamma + emb_beta,
 * and what the first reader makes of them, out[m] = layer_norm(*take * x[m]) * gamma + beta. */
typedef struct b200_rows_start_args {
    const float *emb, *emb_pos; const uint32_t *tokens; int vocab, pos_rows, pos0;
    const float *emb_gamma, *emb_beta, *take, *gamma, *beta; float eps;
    int rows, dim, ld, wtype;
    float *x; void *out;
} b200_rows_start_args;
int b200_rows_start(const b200_rows_start_args *a, void *stream);
/* out[m] = layer norm of x[index[m]] (index NULL: m) times gamma plus beta. */
int b200_rows_layer_norm(const float *x, const int *index, int rows, int dim, int ld, float eps,
                         const float *gamma, const float *beta, int wtype, void *out, void *stream);
/* out[m] = grouped RMS norm of x[index[m]] times gamma; wtype: element type of out (BF16 or F32). */
int b200_rows_norm(const float *x, const int *index, int rows, int dim, int ld, int groups, float eps,
                   const float *gamma, int wtype, void *out, void *stream);
/* out[m][i] = gelu_tanh(gu[m][2i]) * gu[m][2i+1], i < inter; out rows inter elements apart. */
int b200_rows_gelu_mul(const float *gu, long long gu_ld, int rows, int inter, int wtype, void *out, void *stream);
/* x <- cap * tanh(x / cap) over rows of dim floats, ld apart. */
int b200_rows_softcap(float *x, int rows, int dim, long long ld, float cap, void *stream);

/* Last tensor-parallel step of a token: waits for every rank's (value, index)
 * pair, takes the largest (lowest index on ties), stores it as tokens[pos+1]
 * unless that position belongs to the prompt, and advances *pos. */
int b200_tp_argmax_finalize(const float *d_vals, const int *d_idx, int n_ranks,
                            const unsigned *d_wait_flags, const unsigned *d_epoch,
                            int epoch_mul, int epoch_add,
                            int *d_tokens, int *d_pos, const int *d_prompt_len,
                            unsigned *d_epoch_rw, int *d_err, int use_pdl, void *stream);

/* ------------------------------------------------------------------------
 * Whole-token kernel: every matvec and attention step of one token in ONE
 * persistent launch (one block per SM, cooperative). Replaces the reference's
 * single command buffer with its barrier after every dispatch
 * (src/nn/fast_metal.m:223-247; op sequence src/nn/fast_inference.c:394-466).
 *
 * Structure: per layer five stages (q/k/v matvec, attention, o matvec, gate/up
 * matvec, down matvec), then the LM head. A producer warp per block streams
 * the block's share of every stage's weights, in stage order, through one
 * shared-memory ring with bulk copies; it depends on no activation, so it runs
 * ahead across stage boundaries and HBM stays busy while the consumers hand a
 * stage's result over. Hand-over is through "flagged" vectors in global
 * memory: every fp32 value travels as an 8-byte word {value, flag} written
 * with one store, flag = epoch * (n_layers + 1) + layer + 1; a reader polls
 * the word until the flag matches, so data and readiness arrive in the same
 * round trip to L2 and no device-wide barrier exists. The residual stream is
 * kept by every block in its own shared memory and updated from the flagged
 * o / down outputs ("slots", one per tensor-parallel rank, summed in rank
 * order). Every wait is bounded (spin_limit); a wait that runs out raises
 * *d_err and the block's abort flag, after which all later waits fall through.
 *
 * b200_flagged is the 8-byte word: low half the fp32 bits, high half the flag.
 * ---------------------------------------------------------------------- */
typedef unsigned long long b200_flagged;
#define B200_CNT_STRIDE 32
enum { B200_CNT_QKV = 0, B200_CNT_ATTN = 1, B200_CNT_ACT = 2, B200_CNT_SLOTS_O = 3, B200_CNT_SLOTS_DN = 4, B200_CNT_PART = 8 };

/* Pointers of one layer (device table, n_layers entries). Gammas may be NULL where the
 * architecture has none (pre_ff / post_ff outside Gemma3, q/k norm when absent). */
typedef struct b200_token_layer {
    const void *w_qkv, *w_o, *w_gateup, *w_down;     /* packed rows, see the layout note above */
    const float *g_input, *g_post_attn, *g_pre_ff, *g_post_ff, *g_qn, *g_kn;
    /* This layer's rotation for every position: [max_seq][hd/2] pairs (cos, sin) of pos * inv_freq[d], made on
     * the host with the C library's cosf / sinf, i.e. the values the reference's CPU path multiplies with
     * (src/nn/attention.c:757-766). Layers with the same base share one table. */
    const float *rope;
    void *k_cache, *v_cache;                         /* binary16 [n_kv][max_seq][hd] */
} b200_token_layer;

/* Geometry of one matvec stage. rows/cols/row_stride/glu are the caller's; the rest is filled by
 * b200_token_plan. */
typedef struct b200_stage_geom {
    int rows, cols; long long row_stride;
    int glu;                      /* rows are (gate, up) pairs */
    int T, NG, spt;               /* threads per consumer group, groups, 16-byte column slices per thread */
    int rg, rb;                   /* rows per group in a chunk; rows per chunk (one ring slot) = NG * rg */
    int pw;                       /* rows per emission window, a multiple of rb */
    int cta_base, cta_rem;        /* row units per block: base, +1 for the first rem blocks */
    int direct_in;                /* reserved, 0 */
} b200_stage_geom;

enum { B200_ST_QKV = 0, B200_ST_O = 1, B200_ST_GATEUP = 2, B200_ST_DOWN = 3, B200_ST_LM = 4, B200_ST_KINDS = 5 };

typedef struct b200_token_args {
    const b200_token_layer *d_layers; int n_layers;
    int wtype;                                    /* B200_WT_Q8 or B200_WT_F16, all matrices */
    int gemma;                                    /* 1: four-norm block and tanh-GELU (src/nn/fast_inference.c:436-462) */
    b200_stage_geom g[B200_ST_KINDS];
    const void *w_lm; const float *g_final;
    int with_lm;                                  /* 0: stop after the last layer (prompt positions) */
    const float *d_emb; int emb_rows; float emb_scale, eps;
    int d_model, n_q, n_kv, hd, max_seq, n_split;
    /* device control words */
    int *d_pos; int *d_tokens; const int *d_prompt_len; unsigned *d_epoch; int *d_err;
    /* flagged vectors local to this GPU */
    b200_flagged *d_qkv;                          /* [(n_q + 2 n_kv) * hd] */
    b200_flagged *d_attn_part;                    /* [n_q][n_split][hd + 2] */
    b200_flagged *d_attn_out;                     /* [n_q * hd] */
    b200_flagged *d_act;                          /* [g[GATEUP].rows / 2] */
    b200_flagged *d_am;                           /* [2 * blocks]: (best value, row) of each block */
    /* flagged vectors written by every rank: [n_ranks][d_model] each */
    const b200_flagged *d_slots_o, *d_slots_dn;
    b200_flagged *d_peer_slots_o[B200_MAX_PEERS]; /* slot `rank` inside rank p's d_slots_o, p < n_ranks */
    b200_flagged *d_peer_slots_dn[B200_MAX_PEERS];
    const b200_flagged *d_am_rank;                /* [2 * n_ranks] */
    b200_flagged *d_peer_am[B200_MAX_PEERS];      /* entry `rank` inside rank p's d_am_rank */
    int n_ranks, rank;
    /* Arrival counters (hints that spare L2 the polling of 640 threads per block: one thread waits for
     * the count, then everybody reads the flagged words once; the flags stay the proof of validity).
     * Each producer adds the number of words it stored; a reader expects (epoch * n_layers + layer + 1)
     * * words-per-layer. d_counters: B200_CNT_STRIDE words apart: [0] q/k/v rows, [1] attention output,
     * [2] activations, [3] o slots, [4] down slots (all ranks add to these two), [8 + h] partial
     * records of KV head h. Zero-initialised by the caller, never reset. */
    unsigned *d_counters;
    unsigned *d_peer_counters[B200_MAX_PEERS];    /* rank p's d_counters, p < n_ranks */
    float *d_logits; long long logits_offset;     /* logits[logits_offset + r] = row r of this rank's LM-head shard */
    int spin_limit;                               /* iterations of a polling loop before it gives up; 0 = default */
    /* optional trace: 16 words per block and stage, [block][stage][16], 6 stages
     * per layer (q/k/v, attention, o, gate/up, down, one unused) + the LM head: [0] stage entered,
     * [1] input vector complete, [2] first weights in shared memory, [3] thread 0 done with its rows,
     * [4] results stored, [5] producer issued the stage's first copy, [6] its last copy, [7] all warps
     * of the block done with their rows; [8..13] thread 0's first two chunks (data there, rows summed,
     * partials stored), [14] chunks walked, [15] chunks owned. NULL = no trace (a separate kernel instantiation without the
     * timer reads). */
    unsigned long long *d_trace;
    /* filled by b200_token_plan */
    int n_blocks, smem_bytes, scratch_floats;
    int att_keys;                                 /* cache rows the attention stage holds in shared memory at a time */
    /* Bytes of the following stage's weights that a block asks L2 for when it starts streaming a stage
     * (0 = none, the default: the ring alone measured faster on Qwen3-4B). */
    int l2_ahead_bytes;
    /* Iterations one thread per block spends watching an arrival counter before the block polls the flagged
     * words themselves. 0: no counter wait at all, every thread re-reads its own words until their flags
     * match. */
    int counter_spin_limit;
} b200_token_args;

/* Fills the geometry (g[k].T ... direct_in), n_split limits and the launch shape for `n_blocks` blocks
 * (0 = one per SM of the current device). Returns 0, B200_E_BADARG for shapes the kernel does not
 * cover, B200_E_TOOLARGE when a row or the shared-memory budget is exceeded. Host-only arithmetic
 * when n_blocks > 0: callable without a GPU. */
int b200_token_plan(b200_token_args *a, int n_blocks);

/* Host-side replay of the row partition the kernel uses (no GPU needed; for tests): writes up to `cap`
 * triples {first_row, n_rows, window} of block `block`, stage kind `kind`, in the order the producer
 * issues them; returns the number of chunks. */
int b200_token_chunks(const b200_token_args *a, int kind, int block, int *out, int cap);

int b200_decode_token(const b200_token_args *a, void *stream);

/* LoRA side path of one decode token: qkv[0..q_rows) += scaling * B_q (A_q x) and
 * qkv[q_rows + kv_rows ..) += scaling * B_v (A_v x), with x [d_model] the normalised
 * layer input (b200_matvec_args.d_in_copy), A [rank, d_model], B [rows, rank],
 * fp32. Replaces the six per-layer dispatches of src/nn/fast_inference.c:406-421. */
int b200_lora_decode(const float *x, const float *A_q, const float *B_q, const float *A_v, const float *B_v,
                     float *qkv, int d_model, int q_rows, int kv_rows, int rank, float scaling, void *stream);

/* Batched decode: arg-max of each of n_rows logit rows (lowest index on ties,
 * src/nn/fast_inference.c:469-476) written to next_tokens[row] and, when ctl[2]
 * is set, to history[ctl[1]*n_rows + row]; the last row to finish then advances
 * the position ctl[0] (and the step count ctl[1] when recording). done_count is
 * a zeroed scratch word. */
int b200_argmax_rows(const float *logits, int n_rows, int vocab, unsigned *next_tokens, unsigned *history,
                     int max_steps, int *ctl, unsigned *done_count, void *stream);

/* Number of kernel launches issued through this ABI since the last reset
 * (what bench.py reports as gpu_launches). */
unsigned long long b200_launch_count(int reset);
/* For callers that replay captured launches (a CUDA graph): adds the kernel nodes of a replay to the count. */
void b200_launch_count_add(unsigned long long n);

#ifdef __cplusplus
}
#endif
#endif /* LLMB200_KERNELS_H */
