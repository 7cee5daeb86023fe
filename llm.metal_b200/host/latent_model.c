/*
 * Morilorn: a decoder whose layers mix tokens with windowed latent attention (one low-rank cached vector per
 * token and layer), gate each sublayer's result element by element, normalise after the scaled residual sum in
 * groups, and hand on a learned average over all earlier layers' results.
 *
 *   X_0 = scale_e * embed[token],  x = X_0
 *   layer i:  u = norm1(alpha x + sigmoid(W_rg1 x + b1) * mixer(x))
 *             X_{i+1} = norm2(alpha u + sigmoid(W_rg2 u + b2) * W_down(gelu(W_gate u) * W_up u))     (u without a feed-forward)
 *             x = sum_{j <= i+1} dwa_i[j] X_j
 *   logits = cap * tanh(head norm(x) / cap)
 *
 * This file holds the model's weights and enqueues its kernels; state, graphs, generate loop and measurement are
 * the engine's (decode_engine.c). Two paths over the same weights and cache:
 *
 *   one token   seven launches per layer, chained by programmatic dependent launch inside the engine's per-token
 *               graph. Products of the same input are one matrix (q | latent | output gate | residual gate; gate/up
 *               pairs | residual gate). The norm after a sublayer runs in the input assembly of the next product,
 *               the gated residual sum and the part of the depth average that is already known in the output of
 *               the o / down product.
 *   rows        a portion of several tokens, up to ROW_CHUNK at a time: the same matrices as tensor-core products
 *               (fp32: CUDA-core products) with row kernels in between.
 *
 * Layouts: llmb200_up8(n) = n rounded up to a multiple of 8. Matrices get zero padding columns up to llmb200_up8(cols) and sections
 * of fused matrices zero padding rows up to llmb200_up8(rows), vectors zero padding to match, so every size works.
 */
#include "model_dir.h"
#include "../../include/llmb200_train_kernels.h"

#include <math.h>
#include <stdlib.h>
#include <string.h>

typedef struct {
    int heads, dim, rot_dim, rot_dims, vdim, kv_rank, window, ff;
    float scale;
    double rot_base;
    PackedMat in, uk_t, kv, o, gu, down;
    int o_dkv, o_gate, o_rg1;        /* row offsets in `in`; q is at 0 */
    int ffp;                         /* llmb200_up8(ff): gate/up pairs 0 .. 2 ffp, residual gate after them */
    float *dkv_gamma, *norm1, *norm2, *b1, *b2, *dwa;
    const float *rope;
    void *cache;                     /* [max_seq][llmb200_up8(kv_rank) + llmb200_up8(rot_dim)] */
    int n_split;
} LLayer;

typedef struct {
    LLayer *layers;
    int Dp, groups, es;              /* es: bytes of a matrix / cache element */
    float eps, alpha, softcap;
    PackedMat head;
    float **rope_tab; int n_rope;
    /* one token */
    void *qlat;
    float *proj, *part, *attn, *z, *u, *rg2, *act, *hist, *mix, *x;
    /* rows (allocated at the first portion) */
    RowPath rows;
    float *r_proj, *r_hist, *r_x, *r_u, *r_y, *r_gu;
    void *r_xh, *r_q, *r_kv, *r_attn, *r_act;
} Latent;

static int imax(int a, int b) { return a > b ? a : b; }

/* ------------------------------------------------------------ loading */

/* (cos, sin) of pos * base^(-2i/dims), formed in double; one table per distinct (base, dims). */
static const float *rope_table(InferenceState *s, Latent *m, int layer)
{
    LLayer *y = &m->layers[layer];
    for (int i = 0; i < layer; ++i)
        if (m->layers[i].rot_base == y->rot_base && m->layers[i].rot_dims == y->rot_dims) return m->layers[i].rope;
    const int half = y->rot_dims / 2;
    const size_t n = (size_t)s->max_seq * imax(half, 1) * 2;
    float *h = malloc(n * sizeof(float));
    if (!h) return NULL;
    for (int i = 0; i < half; ++i) {
        const double f = pow(y->rot_base, -2.0 * i / y->rot_dims);
        for (int p = 0; p < s->max_seq; ++p) {
            h[((size_t)p * half + i) * 2] = (float)cos(p * f);
            h[((size_t)p * half + i) * 2 + 1] = (float)sin(p * f);
        }
    }
    float *d = llmb200_upload_f32(h, half ? n : 0);
    free(h);
    if (d) m->rope_tab[m->n_rope++] = d;
    return d;
}

static int load_layer(InferenceState *s, Latent *m, int li, const llmb200_tensor_file *file)
{
    LLayer *y = &m->layers[li];
    TensorSource src = { file, li, 0 };
    const int D = s->D, H = y->heads, R = y->kv_rank, dim8 = llmb200_up8(y->dim), vd8 = llmb200_up8(y->vdim), per = dim8 + vd8;
    const int q_rows = H * (y->dim + y->rot_dim), hv = H * y->vdim;
    y->o_dkv = llmb200_up8(q_rows);
    y->o_gate = y->o_dkv + llmb200_up8(R + y->rot_dim);
    y->o_rg1 = y->o_gate + llmb200_up8(hv);
    if (llmb200_new_mat(s, &y->in, y->o_rg1 + m->Dp, D) || llmb200_new_mat(s, &y->uk_t, H * R, y->dim) || llmb200_new_mat(s, &y->kv, H * per, R) ||
        llmb200_new_mat(s, &y->o, D, hv))
        return -1;
    llmb200_load_rows(s, &src, &y->in, "mix.q", q_rows, D, 0, 1);
    llmb200_load_rows(s, &src, &y->in, "mix.dkv", R + y->rot_dim, D, y->o_dkv, 1);
    llmb200_load_rows(s, &src, &y->in, "mix.g", hv, D, y->o_gate, 1);
    llmb200_load_rows(s, &src, &y->in, "rg1", D, D, y->o_rg1, 1);
    llmb200_load_rows(s, &src, &y->o, "mix.o", D, hv, 0, 1);

    /* the two expansions: side by side per head for the rows path, W_uk transposed per head for one token */
    float *uk = llmb200_source_tensor(&src, "mix.uk", (long long)H * y->dim, R), *uv = llmb200_source_tensor(&src, "mix.uv", hv, R);
    float *t = malloc((size_t)R * y->dim * sizeof(float));
    if (uk && uv && t)
        for (int h = 0; h < H && !src.failed; ++h) {
            const float *k = uk + (size_t)h * y->dim * R;
            for (int d = 0; d < y->dim; ++d)
                for (int r = 0; r < R; ++r) t[(size_t)r * y->dim + d] = k[(size_t)d * R + r];
            if (llmb200_put_rows(s, &y->uk_t, t, R, y->dim, h * R, 1) || llmb200_put_rows(s, &y->kv, k, y->dim, R, h * per, 1) ||
                llmb200_put_rows(s, &y->kv, uv + (size_t)h * y->vdim * R, y->vdim, R, h * per + dim8, 1))
                src.failed = 1;
        }
    free(uk); free(uv); free(t);

    y->dkv_gamma = llmb200_load_vec(&src, "mix.dkv.norm", R, llmb200_up8(R));
    y->norm1 = llmb200_load_vec(&src, "norm1", D, m->Dp);
    y->b1 = llmb200_load_vec(&src, "rg1.b", D, m->Dp);
    y->dwa = llmb200_load_vec(&src, "dwa", li + 2, li + 2);
    if (y->ff) {
        y->ffp = llmb200_up8(y->ff);
        if (llmb200_new_mat(s, &y->gu, 2 * y->ffp + m->Dp, D) || llmb200_new_mat(s, &y->down, D, y->ff)) return -1;
        llmb200_load_rows(s, &src, &y->gu, "mlp.gate", y->ff, D, 0, 2);
        llmb200_load_rows(s, &src, &y->gu, "mlp.up", y->ff, D, 1, 2);
        llmb200_load_rows(s, &src, &y->gu, "rg2", D, D, 2 * y->ffp, 1);
        llmb200_load_rows(s, &src, &y->down, "mlp.down", D, y->ff, 0, 1);
        y->norm2 = llmb200_load_vec(&src, "norm2", D, m->Dp);
        y->b2 = llmb200_load_vec(&src, "rg2.b", D, m->Dp);
    }
    const size_t row = (size_t)(llmb200_up8(R) + llmb200_up8(y->rot_dim)) * m->es;
    y->cache = llmb200_dev_zero(row * s->max_seq);
    y->rope = rope_table(s, m, li);
    y->n_split = b200_latent_splits(H, y->window, s->max_seq);
    if (src.failed || !t || !y->cache || !y->rope) return -1;
    const PackedMat *w[] = { &y->in, &y->uk_t, &y->kv, &y->o, &y->gu, &y->down };
    for (int i = 0; i < 6; ++i) {
        const unsigned long long bytes = (unsigned long long)w[i]->stride * w[i]->rows;
        s->weight_bytes += w[i] == &y->kv ? bytes / per * vd8 : bytes;      /* one token reads only the value half of kv */
    }
    return 0;
}

static int parse_layer(const json *e, int i, LLayer *y)
{
    char where[32];
    snprintf(where, sizeof(where), "layer %d", i);
    const char *type = json_string(e, "type");
    if (!type || strcmp(type, "latent_attention")) return llmb200_bad_config(where, "the mixer type is not latent_attention");
    const json *x = json_get(e, "mixer"), *rot = json_get(x, "rot"), *mask = json_get(x, "mask"), *mlp = json_get(e, "mlp");
    double scale;
    if (json_int(x, "heads", &y->heads) || json_int(x, "dim", &y->dim) || json_int(x, "rot_dim", &y->rot_dim) ||
        json_int(x, "vdim", &y->vdim) || json_int(x, "kv_rank", &y->kv_rank) || json_number(x, "scale", &scale) ||
        json_number(rot, "base", &y->rot_base))
        return llmb200_bad_config(where, "a size or constant of the mixer is missing");
    y->scale = (float)scale;
    if (json_int(rot, "dims", &y->rot_dims)) y->rot_dims = y->rot_dim;
    if (mask && mask->type != JSON_NULL && (json_int(mask, "size", &y->window) || y->window < 1))
        return llmb200_bad_config(where, "mask.size must be a positive integer");
    if (y->heads < 1 || y->dim < 1 || y->rot_dim < 1 || y->vdim < 1 || y->kv_rank < 1 || y->rot_dims < 0 || y->rot_dims > y->rot_dim ||
        y->rot_dims % 2 || !(y->rot_base > 0))
        return llmb200_bad_config(where, "a size of the mixer is out of range");
    if (mlp && mlp->type != JSON_NULL) {
        const char *kind = json_string(mlp, "kind");
        if (!kind || strcmp(kind, "dense")) return llmb200_bad_config(where, "the feed-forward kind is not dense");
        if (json_int(mlp, "ff", &y->ff) || y->ff < 1) return llmb200_bad_config(where, "mlp.ff must be a positive integer");
    }
    return 0;
}

static int enqueue_token(InferenceState *s, int with_lm, int pdl);
static int forward_rows(InferenceState *s, const uint32_t *tokens, int n, const int *want, int n_want, float *logits);
static void free_model(InferenceState *s);
static const ModelOps morilorn_ops = { .enqueue_token = enqueue_token, .forward_rows = forward_rows, .free_model = free_model };

static int parse(InferenceState *s, Latent *m, const json *c)
{
    const json *norm = json_get(c, "norm"), *layers = json_get(c, "layers");
    double eps, alpha, emb, cap = 0.0;
    if (json_int(c, "vocab", &s->V) || json_int(c, "width", &s->D) || json_number(norm, "eps", &eps) ||
        json_number(c, "postln_alpha", &alpha) || json_number(json_get(c, "embedding"), "scale", &emb))
        return llmb200_bad_config("model", "a size or constant is missing");
    if (json_int(norm, "groups", &m->groups)) m->groups = 1;
    json_number(c, "logit_softcap", &cap);
    if (s->V < 1 || s->D < 1 || m->groups < 1 || s->D % m->groups) return llmb200_bad_config("model", "a size is out of range");
    if (!layers || layers->type != JSON_ARRAY || layers->n < 1) return llmb200_bad_config("model", "layers must be a list");
    m->eps = (float)eps; m->alpha = (float)alpha; m->softcap = (float)cap;
    s->emb_scale = (float)emb;
    s->L = layers->n;
    m->layers = calloc((size_t)s->L, sizeof(LLayer));
    m->rope_tab = calloc((size_t)s->L, sizeof(float *));
    if (!m->layers || !m->rope_tab) return -1;
    int i = 0;
    for (const json *e = layers->child; e; e = e->next, ++i)
        if (parse_layer(e, i, &m->layers[i]) != 0) return -1;
    return 0;
}

InferenceState *llmb200_create_morilorn(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype)
{
    Latent *m = calloc(1, sizeof(*m));
    InferenceState *s = m ? llmb200_dir_state(&morilorn_ops, MODEL_MORILORN, m, max_seq_len, wtype) : NULL;
    if (!s) return NULL;
    if (parse(s, m, config) != 0) goto fail;
    m->es = wtype == B200_WT_F32 ? 4 : 2;
    m->Dp = llmb200_up8(s->D);
    s->V_l = s->V;

    int proj = 0, qlat = 0, part = 0, attn = 0, act = 8;
    for (int i = 0; i < s->L; ++i) {
        if (load_layer(s, m, i, tensors) != 0) { fprintf(stderr, "[FastGen] loading layer %d failed\n", i); goto fail; }
        const LLayer *y = &m->layers[i];
        proj = imax(proj, y->in.rows);
        qlat = imax(qlat, y->heads * (llmb200_up8(y->kv_rank) + llmb200_up8(y->rot_dim)));
        part = imax(part, y->heads * y->n_split * (llmb200_up8(y->kv_rank) + 8));
        attn = imax(attn, y->o.cols);
        act = imax(act, y->ffp);
    }
    TensorSource src = { tensors, -1, 0 };
    if (llmb200_new_mat(s, &m->head, s->V, s->D) != 0) goto fail;
    llmb200_load_rows(s, &src, &m->head, "head", s->V, s->D, 0, 1);
    s->weight_bytes += (unsigned long long)m->head.stride * s->V;
    s->g_final = llmb200_load_vec(&src, "final.norm", s->D, m->Dp);
    s->emb = llmb200_load_table(&src, "embed", s->V, s->D, m->Dp);
    if (src.failed) goto fail;

    m->proj = llmb200_dev_zero((size_t)proj * 4); m->qlat = llmb200_dev_zero((size_t)qlat * 4);
    m->part = llmb200_dev_zero((size_t)part * 4); m->attn = llmb200_dev_zero((size_t)attn * 4);
    m->act = llmb200_dev_zero((size_t)act * 4); m->rg2 = llmb200_dev_zero((size_t)imax(64, m->Dp) * 4);
    m->z = llmb200_dev_zero((size_t)2 * m->Dp * 4); m->u = llmb200_dev_zero((size_t)m->Dp * 4);
    m->mix = llmb200_dev_zero((size_t)m->Dp * 4); m->x = llmb200_dev_zero((size_t)m->Dp * 4);
    m->hist = llmb200_dev_zero((size_t)(s->L + 1) * m->Dp * 4);
    if (!m->proj || !m->qlat || !m->part || !m->attn || !m->act || !m->rg2 || !m->z || !m->u || !m->mix || !m->x || !m->hist) goto fail;
    if (llmb200_engine_common(s) != 0 || cudaStreamSynchronize(g_rt.stream) != cudaSuccess) goto fail;
    s->finished = 1;
    return s;
fail:
    inference_state_free(s);
    return NULL;
}

static void free_model(InferenceState *s)
{
    Latent *m = s->model;
    if (!m) return;
    for (int i = 0; m->layers && i < s->L; ++i) {
        LLayer *y = &m->layers[i];
        void *b[] = { y->in.w, y->uk_t.w, y->kv.w, y->o.w, y->gu.w, y->down.w, y->dkv_gamma, y->norm1, y->norm2, y->b1, y->b2, y->dwa, y->cache };
        for (size_t k = 0; k < sizeof(b) / sizeof(b[0]); ++k) cudaFree(b[k]);
    }
    for (int i = 0; i < m->n_rope; ++i) cudaFree(m->rope_tab[i]);
    void *b[] = { m->head.w, m->proj, m->qlat, m->part, m->attn, m->z, m->u, m->rg2, m->act, m->hist, m->mix, m->x, m->r_proj, m->r_hist,
                  m->r_x, m->r_u, m->r_y, m->r_gu, m->r_xh, m->r_q, m->r_kv, m->r_attn, m->r_act };
    for (size_t k = 0; k < sizeof(b) / sizeof(b[0]); ++k) cudaFree(b[k]);
    llmb200_row_path_free(&m->rows);
    free(m->layers);
    free(m->rope_tab);
    free(m);
    s->model = NULL;
}

/* ------------------------------------------------------------ one token */

static void latent_args(InferenceState *s, const Latent *m, const LLayer *y, const float *proj, b200_latent_args *a)
{
    memset(a, 0, sizeof(*a));
    a->wtype = s->wtype;
    a->heads = y->heads; a->dim = y->dim; a->rot_dim = y->rot_dim; a->rot_dims = y->rot_dims; a->vdim = y->vdim;
    a->kv_rank = y->kv_rank; a->window = y->window; a->max_seq = s->max_seq;
    a->scale = y->scale; a->eps = m->eps;
    a->d_q = proj; a->d_dkv = proj + y->o_dkv; a->d_gate = proj + y->o_gate;
    a->d_dkv_gamma = y->dkv_gamma; a->d_rope = y->rope; a->d_cache = y->cache;
    a->d_w_uk_t = y->uk_t.w; a->d_w_kv = y->kv.w;
}

static void base(InferenceState *s, const Latent *m, b200_matvec_args *a, const PackedMat *w, int rows, int pdl)
{
    llmb200_matvec_base(s, a, w, m->eps, pdl);
    a->rows = rows;
    a->norm_dim = s->D; a->norm_groups = m->groups;
    a->n_out = 1;
}

/* x = (depth sum of the older results) + coefficient * norm(z), z being what layer l left */
static void take_layer_result(const Latent *m, int l, const float *z, b200_matvec_args *a)
{
    const LLayer *y = &m->layers[l];
    a->in_mode = B200_IN_POSTNORM;
    a->d_in_vec = z;
    a->d_slot_norm_gamma = y->ff ? y->norm2 : y->norm1;
    a->d_mix_in = m->mix; a->d_mix_coef = y->dwa + l + 1;
}

/* z = alpha * resid + sigmoid(gate + bias) * y, and for a layer's last product the depth sum over X_0 .. X_l */
static void gated(const Latent *m, int l, int last, const float *resid, const float *gate, const float *bias, float *z, b200_matvec_args *a)
{
    a->in_mode = B200_IN_VEC;
    a->norm_dim = a->norm_groups = 0;                        /* this product's input is not of the model's width */
    a->out_mode = B200_OUT_GATED;
    a->d_out_resid = resid; a->d_out_gate = gate; a->d_out_gate_bias = bias; a->resid_alpha = m->alpha;
    a->d_out[0] = z;
    if (last) {
        a->d_hist = m->hist; a->hist_n = l + 1; a->hist_stride = m->Dp;
        a->d_hist_coef = m->layers[l].dwa; a->d_hist_out = m->mix;
    }
}

static int enqueue_token(InferenceState *s, int with_lm, int pdl)
{
    const Latent *m = s->model;
    const int D = s->D, L = s->L, Dp = m->Dp;
    void *st = g_rt.stream;
    float *z1 = m->z, *z2 = m->z + Dp;
    b200_matvec_args a;
    for (int l = 0; l < L; ++l) {
        const LLayer *y = &m->layers[l];
        const float *x = l ? m->x : m->hist;
        const int end_at_o = !with_lm && l == L - 1 && !y->ff, end_at_down = !with_lm && l == L - 1 && y->ff;
        /* --- q | latent | gates of this layer's input --- */
        base(s, m, &a, &y->in, y->o_rg1 + Dp, pdl);
        if (l == 0) {
            a.in_mode = B200_IN_EMBED; a.d_emb = s->emb; a.d_tokens = s->d_tokens; a.emb_scale = s->emb_scale; a.emb_rows = s->V;
            a.d_resid_out = m->hist;                          /* X_0 */
        } else {
            take_layer_result(m, l - 1, m->layers[l - 1].ff ? z2 : z1, &a);
            a.d_post_copy = m->hist + (size_t)l * Dp;         /* X_l */
            a.d_resid_out = m->x;
        }
        a.out_mode = B200_OUT_STORE; a.d_out[0] = m->proj;
        llmb200_prof_mark(s, K_QKV);
        if (llmb200_want_kind(s, K_QKV, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
        /* --- attention --- */
        b200_latent_args at;
        latent_args(s, m, y, m->proj, &at);
        at.d_qlat = m->qlat; at.d_part = m->part; at.d_out = m->attn; at.d_pos = s->d_pos;
        at.n_split = y->n_split; at.use_pdl = pdl;
        llmb200_prof_mark(s, K_ATTN);
        if (llmb200_want_kind(s, K_ATTN, NULL)) K_TRY(b200_latent_decode(&at, st), return -1);
        llmb200_prof_mark(s, -1);
        /* --- o, gated residual sum --- */
        base(s, m, &a, &y->o, D, pdl);
        a.d_in_vec = m->attn;
        gated(m, l, !y->ff, x, m->proj + y->o_rg1, y->b1, z1, &a);
        if (end_at_o) { a.d_ticket = s->mv_ticket; a.advance_pos = 1; a.advance_epoch = 1; }
        llmb200_prof_mark(s, K_O);
        if (llmb200_want_kind(s, K_O, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
        if (!y->ff) continue;
        /* --- norm, gate/up | residual gate --- */
        base(s, m, &a, &y->gu, 2 * y->ffp + Dp, pdl);
        a.in_mode = B200_IN_POSTNORM; a.d_in_vec = z1; a.d_slot_norm_gamma = y->norm1; a.d_resid_out = m->u;
        a.out_mode = B200_OUT_GLU; a.act = 1; a.glu_rows = 2 * y->ffp; a.d_out[0] = m->act; a.d_out2 = m->rg2;
        llmb200_prof_mark(s, K_GATEUP);
        if (llmb200_want_kind(s, K_GATEUP, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
        /* --- down, gated residual sum --- */
        base(s, m, &a, &y->down, D, pdl);
        a.d_in_vec = m->act;
        gated(m, l, 1, m->u, m->rg2, y->b2, z2, &a);
        if (end_at_down) { a.d_ticket = s->mv_ticket; a.advance_pos = 1; a.advance_epoch = 1; }
        llmb200_prof_mark(s, K_DOWN);
        if (llmb200_want_kind(s, K_DOWN, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
    }
    if (!with_lm) return 0;
    base(s, m, &a, &m->head, s->V, pdl);
    take_layer_result(m, L - 1, m->layers[L - 1].ff ? z2 : z1, &a);
    a.d_norm_gamma = s->g_final;
    a.out_mode = B200_OUT_STORE; a.d_out[0] = (float *)(s->comm + s->off_logits); a.softcap = m->softcap;
    a.d_ticket = s->mv_ticket; a.d_argmax_scratch = s->am_scratch;
    a.n_argmax_out = 1;
    a.d_argmax_val[0] = (float *)(s->comm + s->off_am_val); a.d_argmax_idx[0] = (int *)(s->comm + s->off_am_idx);
    a.d_next_token = s->d_tokens; a.d_prompt_len = s->d_prompt_len; a.advance_pos = 1; a.advance_epoch = 1;
    llmb200_prof_mark(s, K_LM);
    if (llmb200_want_kind(s, K_LM, &a)) K_TRY(b200_matvec(&a, st), return -1);
    llmb200_prof_mark(s, -1);
    return 0;
}

/* ------------------------------------------------------------ rows */

static int rows_ready(InferenceState *s, Latent *m)
{
    if (m->rows.chunk) return 0;
    const int M = llmb200_row_chunk(s), Dp = m->Dp, es = m->es;
    size_t proj = 0, q = 0, kv = 0, attn = 0, gu = 0, act = 0;
    for (int i = 0; i < s->L; ++i) {
        const LLayer *y = &m->layers[i];
#define MAXI(v, n) do { const size_t n__ = (size_t)(n); if (n__ > v) v = n__; } while (0)
        long long span = y->window > 0 ? (long long)M + y->window - 1 : s->max_seq;
        if (span > s->max_seq) span = s->max_seq;
        MAXI(proj, y->in.rows);
        MAXI(q, y->heads * (llmb200_up8(y->dim) + llmb200_up8(y->rot_dim)));
        MAXI(kv, span * y->kv.rows);
        MAXI(attn, y->o.cols);
        if (y->ff) { MAXI(gu, y->gu.rows); MAXI(act, y->ffp); }
#undef MAXI
    }
    m->r_proj = llmb200_dev_zero(M * proj * 4); m->r_hist = llmb200_dev_zero((size_t)(s->L + 1) * M * Dp * 4);
    m->r_x = llmb200_dev_zero((size_t)M * Dp * 4); m->r_u = llmb200_dev_zero((size_t)M * Dp * 4);
    m->r_y = llmb200_dev_zero((size_t)M * imax(64, Dp) * 4); m->r_gu = llmb200_dev_zero(M * gu * 4);
    m->r_xh = llmb200_dev_zero((size_t)M * Dp * 2); m->r_q = llmb200_dev_zero(M * q * es); m->r_kv = llmb200_dev_zero(kv * es);
    m->r_attn = llmb200_dev_zero(M * attn * es); m->r_act = llmb200_dev_zero(M * act * es);
    if (!m->r_proj || !m->r_hist || !m->r_x || !m->r_u || !m->r_y || !m->r_gu || !m->r_xh || !m->r_q || !m->r_kv || !m->r_attn || !m->r_act)
        return -1;
    return llmb200_row_path_ready(s, &m->rows, &m->head, Dp, M);
}

/* M tokens from position pos0 on, whose ids are in d_tokens; x of the last layer is left in r_x. */
static int chunk_rows(InferenceState *s, int pos0, int M)
{
    Latent *m = s->model;
    const int Dp = m->Dp, f32 = s->wtype == B200_WT_F32;
    const size_t hs = (size_t)m->rows.chunk * Dp;                 /* one layer's result of a chunk in r_hist */
    void *st = g_rt.stream;
    /* the operand of a product is the bfloat16 copy, or the vector itself in fp32 */
    void *xh = f32 ? NULL : m->r_xh;
    K_TRY(b200_rows_embed(s->emb, (const uint32_t *)s->d_tokens + pos0, M, s->V, Dp, s->emb_scale, m->r_hist, xh, st), return -1);
    for (int l = 0; l < s->L; ++l) {
        const LLayer *y = &m->layers[l];
        const float *x = l ? m->r_x : m->r_hist;
        const long long pld = y->in.rows;
        if (llmb200_rows_product(s, f32 ? (const void *)x : xh, Dp, &y->in, M, m->r_proj, pld, NULL, 0)) return -1;

        b200_latent_args at;
        latent_args(s, m, y, m->r_proj, &at);
        at.n_rows = M; at.pos0 = pos0; at.proj_ld = pld;
        at.kv_row0 = y->window > 0 && pos0 - y->window + 1 > 0 ? pos0 - y->window + 1 : 0;
        at.d_q_rows = m->r_q; at.d_kv = m->r_kv; at.kv_ld = y->kv.rows;
        at.d_out_rows = m->r_attn; at.out_ld = y->o.cols;
        K_TRY(b200_latent_rows_prep(&at, st), return -1);
        const long long cs = llmb200_up8(y->kv_rank) + llmb200_up8(y->rot_dim);
        if (llmb200_rows_product(s, (const char *)y->cache + (size_t)at.kv_row0 * cs * m->es, cs, &y->kv, pos0 + M - at.kv_row0, NULL, y->kv.rows, m->r_kv, 0))
            return -1;
        K_TRY(b200_latent_rows_attend(&at, st), return -1);
        if (llmb200_rows_product(s, m->r_attn, y->o.cols, &y->o, M, m->r_y, y->o.rows, NULL, 0)) return -1;

        b200_rows_postnorm_args pn;
        memset(&pn, 0, sizeof(pn));
        pn.rows = M; pn.dim = s->D; pn.ld = Dp; pn.groups = m->groups; pn.alpha = m->alpha; pn.eps = m->eps;
        pn.y = m->r_y; pn.y_ld = y->o.rows;
        pn.x = x; pn.gate = m->r_proj + y->o_rg1; pn.gate_ld = pld; pn.gate_bias = y->b1; pn.gamma = y->norm1;
        pn.out_h = xh;
        if (y->ff) {
            pn.norm_out = m->r_u; pn.out = m->r_u;
            K_TRY(b200_rows_postnorm(&pn, st), return -1);
            if (llmb200_rows_product(s, f32 ? (const void *)m->r_u : xh, Dp, &y->gu, M, m->r_gu, y->gu.rows, NULL, 0)) return -1;
            K_TRY(b200_rows_gelu_mul(m->r_gu, y->gu.rows, M, y->ffp, s->wtype, m->r_act, st), return -1);
            if (llmb200_rows_product(s, m->r_act, y->ffp, &y->down, M, m->r_y, y->down.rows, NULL, 0)) return -1;
            pn.y_ld = y->down.rows;
            pn.x = m->r_u; pn.gate = m->r_gu + 2 * y->ffp; pn.gate_ld = y->gu.rows; pn.gate_bias = y->b2; pn.gamma = y->norm2;
        }
        pn.norm_out = m->r_hist + (size_t)(l + 1) * hs;
        pn.hist = m->r_hist; pn.hist_n = l + 1; pn.hist_stride = (long long)hs; pn.coef = y->dwa;
        pn.out = m->r_x;
        K_TRY(b200_rows_postnorm(&pn, st), return -1);
    }
    return 0;
}

static int last_rows(InferenceState *s, const int *index, int n, void *out)
{
    const Latent *m = s->model;
    K_TRY(b200_rows_norm(m->r_x, index, n, s->D, m->Dp, m->groups, m->eps, s->g_final, s->wtype, out, g_rt.stream), return -1);
    return 0;
}

static int forward_rows(InferenceState *s, const uint32_t *tokens, int n, const int *want, int n_want, float *logits)
{
    Latent *m = s->model;
    if (rows_ready(s, m) != 0) { fprintf(stderr, "[FastGen] no memory for the row path\n"); return -1; }
    return llmb200_row_path_run(s, &m->rows, chunk_rows, last_rows, m->softcap, tokens, n, want, n_want, logits);
}
