/* The engine's state and the helpers that the model types share (internal). */
#ifndef LLMB200_ENGINE_H
#define LLMB200_ENGINE_H

#include "internal.h"
#include "../../include/llmb200_inference.h"
#include "../../include/llmb200_sft.h"

typedef struct { void *w; long long stride; int rows, cols; } PackedMat;

typedef struct {
    PackedMat qkv, o, gateup, down;
    float *g_input, *g_post_attn, *g_pre_ff, *g_post_ff, *g_qn, *g_kn;
    float *inv_freq;
    float rope_theta;
    const float *rope;       /* this layer's table in InferenceState.rope_tab (whole-token kernel) */
    void *k_cache, *v_cache;
    int loaded;
} Layer;

enum { K_QKV = 0, K_ATTN, K_O, K_GATEUP, K_DOWN, K_LM, K_KINDS };

/* The generate loop lets forwards run ahead of the ids it has read: ids are read in groups of TOK_BATCH, two groups in
 * flight, and after an end id the forwards already launched are not used. State that is not addressed by position has to
 * reach RUN_AHEAD positions back. */
enum { TOK_BATCH = 4, RUN_AHEAD = 2 * TOK_BATCH };

/* What a model type brings to the engine. The engine owns the control words, the per-token graphs, the generate
 * loop, positions, EOS handling and measurement; a model type enqueues its kernels. */
typedef struct {
    /* Enqueue the kernels of one token (position, id and prompt length are in device memory) on the library
     * stream; with_lm: down to the logits, the greedy pick and the fed-back id. Must advance *d_pos. */
    int (*enqueue_token)(InferenceState *s, int with_lm, int pdl);
    /* Run n tokens (already checked) from position s->cur_len on in one pass over the weights and leave the cache
     * behind them; logits of the tokens want[0..n_want) (ascending places among the n) go to `logits`
     * [n_want][V]. NULL: the model type only has the per-token path. */
    int (*forward_rows)(InferenceState *s, const uint32_t *tokens, int n, const int *want, int n_want, float *logits);
    void (*free_model)(InferenceState *s);
    int whole_token;             /* the whole-token kernel can run this model type */
} ModelOps;

struct InferenceState {
    const ModelOps *ops;
    void *model;                 /* what ops keeps about the model beyond the fields below */
    int D, Hq, Hkv, hd, IS, V, L, max_seq, use_fp16, wtype;
    ModelType mt;
    int tp_rank, tp_size, Hq_l, Hkv_l, IS_l, V_l;
    float emb_scale;
    int eos[4], n_eos;

    Layer *layers;
    PackedMat lm;
    float *g_final, *emb;
    int finished;
    unsigned long long weight_bytes;

    /* activations and scratch (device) */
    float *resid[2], *qkv, *attn_out, *act, *attn_scratch, *am_scratch;
    unsigned *attn_tickets, *mv_ticket;
    int n_split;

    /* control words (device): pos, prompt_len, err, epoch, tokens[max_seq+2] */
    int *d_pos, *d_prompt_len, *d_err, *d_tokens;
    unsigned *d_epoch;

    /* all-reduce region, shared with the peers */
    char *comm;
    size_t comm_bytes, off_slots_o, off_slots_dn, off_flags, off_am_val, off_am_idx, off_logits;
    char *peer[B200_MAX_PEERS];
    int connected, loopback;
    /* single-process tensor parallelism (LLMB200_TP=k): the handle a caller holds is rank 0's state */
    int group_n, group_dev[B200_MAX_PEERS], local_peers;
    struct InferenceState *group[B200_MAX_PEERS];

    /* host side */
    float *h_logits;
    int *h_tok;              /* pinned ring for generated ids */
    int *h_ctl;              /* pinned staging for control writes */
    cudaEvent_t tok_ev[4];
    cudaEvent_t ev_a, ev_b;
    cudaGraphExec_t g_full, g_nolm;
    int kernels_full, kernels_nolm;   /* kernel nodes per graph */
    int use_pdl;
    /* LoRA adapter attached with inference_state_set_lora: device pointers into the SFT state's vectors */
    struct { const float *A_q, *B_q, *A_v, *B_v; } *lora;
    int lora_rank;
    float lora_scaling;
    SFTState *sft_src;                    /* the SFT state whose matrices this state copied, or NULL */
    unsigned long long sft_version;       /* its weights_version at the time of the copy */
    float *xnorm;            /* [D]: the normalised layer input, kept by the q/k/v matvec for the LoRA kernel */
    int cur_len;
    double last_decode_ms, last_prefill_ms;
    int last_n_decoded;

    /* instrumentation */
    cudaEvent_t *prof_ev;
    int prof_n, prof_cap, prof_on;
    /* whole-token kernel: layer table on the device, flagged hand-over vectors, launch arguments */
    b200_token_layer *d_tk_layers;
    float *rope_tab[8];      /* rotation tables, one per distinct RoPE base */
    int n_rope_tab;
    b200_flagged *fl_qkv, *fl_part, *fl_attn, *fl_act, *fl_am;
    size_t off_fl_slots_o, off_fl_slots_dn, off_fl_am, off_counters;
    b200_token_args tk;              /* planned arguments; with_lm is set per launch */
    int fused, tk_planned, n_sm;
    unsigned long long *d_step_ns;   /* stage trace of the whole-token kernel (LLMB200_TRACE=1) */
    int only_kind;           /* >= 0: enqueue_token launches only this kind of kernel (timing loops) */
    int *prof_kind;
};

/* Device memory, zero-filled on the library stream. */
float *llmb200_dev_zero(size_t bytes);
/* What every model type needs beside its weights: control words, logits, host buffers, events. D, V, L, max_seq and
 * the tensor-parallel fields must be set. */
int llmb200_engine_common(InferenceState *s);
/* This process's tensor-parallel rank and size (llmb200_set_tp or the environment). */
void llmb200_engine_tp(int *rank, int *world);
/* Fields common to every matvec launch of a state. */
void llmb200_matvec_base(InferenceState *s, b200_matvec_args *a, const PackedMat *m, float eps, int pdl);
/* Timing loops launch one kind of kernel only: 0 = skip this launch; token-state side effects are taken out of *a. */
int llmb200_want_kind(InferenceState *s, int kind, b200_matvec_args *a);
/* Event before (kind >= 0) and after (kind < 0) the launches of a kind, when a profiling pass is on. */
void llmb200_prof_mark(InferenceState *s, int kind);
/* Writes pos / prompt_len (and, when n_tok > 0, token ids starting at tok_at) into the control block. */
int llmb200_set_control(InferenceState *s, int pos, int prompt_len, const uint32_t *tok, int tok_at, int n_tok);
/* The whole file as a NUL-terminated heap buffer, NULL when it cannot be read. */
char *llmb200_slurp(const char *path);

#endif
