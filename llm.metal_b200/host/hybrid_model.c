/*
 * Zidepel: a decoder whose layers mix tokens with grouped-query attention or gated linear attention, in any order, over
 * several residual streams, with layer norms and learned positions. A range of layers can run several times in a row
 * with the same weights.
 *
 *   X_1 = .. = X_n = x_0 = norm(embed[token] + pos[position])
 *   sublayer (a layer's mixer, then its feed-forward, if any):
 *       y = sublayer(norm(sum_s in[s] X_s)),   X_t <- sum_s mix[s][t] X_s + out[t] y
 *   logits = head norm(sum_s X_s)
 *
 *   attention      queries and keys RMS-normed per head, a per-position query factor, capped scores, no rotation
 *   gla            per head a state that decays per key channel (b200_gla_args)
 *   feed-forward   W_down max(W_up h, 0)^2
 *
 * A "run" is one pass of a layer: it has its own cache or state, and connections of its own, because what the streams
 * hand to the next reader depends on which sublayer comes next. This file holds the weights and enqueues the kernels;
 * the rest is the engine's (decode_engine.c). Two paths over the same weights, caches and states:
 *
 *   one token   three to five launches per run, chained by programmatic dependent launch inside the engine's per-token
 *               graph: the products of one input are one matrix; its layer norm runs in the input assembly, the stream
 *               update and the next reader's combination in the output of the o / down product.
 *   rows        a portion of several tokens: the same matrices as tensor-core products (fp32: CUDA-core products) with
 *               row kernels in between.
 *
 * Matrices get zero padding columns up to up8(cols) and sections of fused matrices zero padding rows up to up8(rows),
 * vectors zero padding to match, so every size works.
 */
#include "model_dir.h"
#include "../../include/llmb200_train_kernels.h"

#include <math.h>
#include <stdlib.h>
#include <string.h>

#define up8 llmb200_up8

enum { STATE_SLOTS = RUN_AHEAD + 1, CHUNK = B200_GLA_CHUNK };
enum { MIX_ATTENTION, MIX_GLA };

typedef struct {
    int mixer, heads, kv_heads, dim, vdim, rank, ff;
    float scale, softcap, tau;
    double temp_coef, temp_every;            /* temp_every 0: no query factor */
    PackedMat in, o, up, down;
    int o_k, o_v, o_g, o_f;                  /* row offsets in `in`; q is at 0 */
    float *norm_w[2], *norm_b[2];            /* before the mixer and the feed-forward */
    float *q_gamma, *k_gamma;
    const float *q_scale;
    float *a2, *a2_bias, *mix_gamma;
    float *take[2], *spread[2], *mix[2];     /* host: what a sublayer reads of the streams, where its result goes, the old ones */
    int n_split;
} HLayer;

typedef struct {
    int layer;
    void *k_cache, *v_cache;                 /* [kv_heads][max_seq] rows */
    float *state;                            /* [STATE_SLOTS][heads][dim][up8(vdim)] */
    float *connect[2];                       /* mix | spread | the next reader's take */
} Run;

typedef struct {
    HLayer *layers; int n_layers;
    Run *runs;                               /* as many as the engine's L */
    int Dp, n_streams, max_positions, es;    /* es: bytes of a matrix / cache element */
    int loop_start, loop_stop, loop_times;
    float eps;
    PackedMat head;
    float *pos, *emb_w, *emb_b, *final_b, *first_take;
    float **tables; int n_tables;            /* query factors */
    /* one token */
    float *proj, *attn, *act, *part, *x0, *streams[2], *u;
    unsigned *tickets;
    /* rows (allocated at the first portion) */
    RowPath rows;
    float *r_proj, *r_x0, *r_streams[2], *r_u, *r_y, *r_decay, *r_o;
    void *r_h, *r_q, *r_attn, *r_act, *r_qd, *r_kd, *r_values, *r_scores, *r_chunk;
} Hybrid;

static size_t smax(size_t a, size_t b) { return a > b ? a : b; }

/* ------------------------------------------------------------ configuration */

static int parse_layer(const json *e, int i, HLayer *y)
{
    char where[32];
    snprintf(where, sizeof(where), "layer %d", i);
    const char *type = json_string(e, "type");
    const json *x = json_get(e, "mixer"), *mlp = json_get(e, "mlp");
    double v = 0.0;
    if (!type) return llmb200_bad_config(where, "the mixer type is missing");
    if (json_int(x, "heads", &y->heads) || json_int(x, "dim", &y->dim) || json_int(x, "vdim", &y->vdim) ||
        y->heads < 1 || y->dim < 1 || y->vdim < 1)
        return llmb200_bad_config(where, "a size of the mixer is missing or out of range");
    if (!strcmp(type, "attention")) {
        y->mixer = MIX_ATTENTION;
        if (json_int(x, "kv_heads", &y->kv_heads) || y->kv_heads < 1 || y->heads % y->kv_heads)
            return llmb200_bad_config(where, "mixer.kv_heads must divide the heads");
        if (json_number(x, "scale", &v)) return llmb200_bad_config(where, "mixer.scale is missing");
        y->scale = (float)v;
        const json *cap = json_get(x, "softcap"), *temp = json_get(x, "q_temp");
        if (cap && cap->type != JSON_NULL) {
            if (json_number(x, "softcap", &v) || !(v > 0.0)) return llmb200_bad_config(where, "mixer.softcap must be positive");
            y->softcap = (float)v;
        }
        if (temp && temp->type != JSON_NULL &&
            (json_number(temp, "coef", &y->temp_coef) || json_number(temp, "every", &y->temp_every) || !(y->temp_every > 0.0)))
            return llmb200_bad_config(where, "mixer.q_temp needs coef and a positive every");
    } else if (!strcmp(type, "gla")) {
        y->mixer = MIX_GLA;
        if (json_number(x, "tau", &v) || !(v > 0.0)) return llmb200_bad_config(where, "mixer.tau must be positive");
        y->tau = (float)v;
    } else return llmb200_bad_config(where, "the mixer type is neither attention nor gla");
    if (mlp && mlp->type != JSON_NULL) {
        const char *kind = json_string(mlp, "kind");
        if (!kind || strcmp(kind, "dense")) return llmb200_bad_config(where, "the feed-forward kind is not dense");
        if (json_int(mlp, "ff", &y->ff) || y->ff < 1) return llmb200_bad_config(where, "mlp.ff must be a positive integer");
    }
    return 0;
}

/* The layers in the order they run, the looped range `times` times over. */
static int make_runs(InferenceState *s, Hybrid *m)
{
    const int span = m->loop_stop - m->loop_start;
    const long long n = m->n_layers + (long long)span * (m->loop_times - 1);
    if (n < 1 || n > 4096) return llmb200_bad_config("loop", "the number of layer runs is out of range");
    m->runs = calloc((size_t)n, sizeof(Run));
    if (!m->runs) return -1;
    s->L = (int)n;
    for (int r = 0; r < s->L; ++r) {
        const int inside = r - m->loop_start, total = span * m->loop_times;
        m->runs[r].layer = inside < 0 ? r : inside < total ? m->loop_start + inside % span : m->loop_stop + inside - total;
    }
    return 0;
}

static int parse(InferenceState *s, Hybrid *m, const json *c)
{
    const json *layers = json_get(c, "layers"), *loop = json_get(c, "loop");
    double eps;
    if (json_int(c, "vocab", &s->V) || json_int(c, "width", &s->D) || json_number(json_get(c, "norm"), "eps", &eps) ||
        json_int(c, "streams", &m->n_streams) || json_int(c, "max_positions", &m->max_positions))
        return llmb200_bad_config("model", "a size or constant is missing");
    if (s->V < 1 || s->D < 1 || m->max_positions < 1) return llmb200_bad_config("model", "a size is out of range");
    if (m->n_streams < 1 || m->n_streams > B200_MAX_STREAMS) return llmb200_bad_config("model", "streams must be 1 to 8");
    if (!layers || layers->type != JSON_ARRAY || layers->n < 1) return llmb200_bad_config("model", "layers must be a list");
    m->eps = (float)eps;
    m->n_layers = layers->n;
    m->layers = calloc((size_t)m->n_layers, sizeof(HLayer));
    m->tables = calloc((size_t)m->n_layers, sizeof(float *));
    if (!m->layers || !m->tables) return -1;
    int i = 0;
    for (const json *e = layers->child; e; e = e->next, ++i)
        if (parse_layer(e, i, &m->layers[i]) != 0) return -1;
    m->loop_times = 1;
    if (loop && loop->type != JSON_NULL &&
        (json_int(loop, "start", &m->loop_start) || json_int(loop, "stop", &m->loop_stop) || json_int(loop, "times", &m->loop_times) ||
         m->loop_start < 0 || m->loop_stop < m->loop_start || m->loop_stop > m->n_layers || m->loop_times < 1))
        return llmb200_bad_config("loop", "needs 0 <= start <= stop <= layers and times >= 1");
    if (s->max_seq > m->max_positions) s->max_seq = m->max_positions;        /* a position past the table does not exist */
    return make_runs(s, m);
}

/* ------------------------------------------------------------ loading */

/* 1 + coef * ln(floor((p + 1) / every) + 1) per position, formed in double; one table per distinct (coef, every). */
static const float *factor_table(InferenceState *s, Hybrid *m, int layer)
{
    HLayer *y = &m->layers[layer];
    for (int i = 0; i < layer; ++i)
        if (m->layers[i].q_scale && m->layers[i].temp_coef == y->temp_coef && m->layers[i].temp_every == y->temp_every) return m->layers[i].q_scale;
    float *h = malloc((size_t)s->max_seq * sizeof(float));
    if (!h) return NULL;
    for (int p = 0; p < s->max_seq; ++p) h[p] = (float)(1.0 + y->temp_coef * log(floor((p + 1) / y->temp_every) + 1.0));
    float *d = llmb200_upload_f32(h, (size_t)s->max_seq);
    free(h);
    if (d) m->tables[m->n_tables++] = d;
    return d;
}

static int load_sublayer(Hybrid *m, HLayer *y, TensorSource *src, int q, int D)
{
    char name[32];
    const int n = m->n_streams;
    snprintf(name, sizeof(name), "norm%d", q + 1);   y->norm_w[q] = llmb200_load_vec(src, name, D, m->Dp);
    snprintf(name, sizeof(name), "norm%d.b", q + 1); y->norm_b[q] = llmb200_load_vec(src, name, D, m->Dp);
    snprintf(name, sizeof(name), "hc%d.in", q + 1);  y->take[q] = llmb200_source_tensor(src, name, n, 0);
    snprintf(name, sizeof(name), "hc%d.out", q + 1); y->spread[q] = llmb200_source_tensor(src, name, n, 0);
    snprintf(name, sizeof(name), "hc%d.mix", q + 1); y->mix[q] = llmb200_source_tensor(src, name, n, n);
    return src->failed ? -1 : 0;
}

static int load_layer(InferenceState *s, Hybrid *m, int li, const llmb200_tensor_file *file)
{
    HLayer *y = &m->layers[li];
    TensorSource src = { file, li, 0 };
    const int D = s->D, qk = y->heads * y->dim, hv = y->heads * y->vdim;
    int rows;
    if (y->mixer == MIX_ATTENTION) {
        y->o_k = up8(qk);
        y->o_v = y->o_k + up8(y->kv_heads * y->dim);
        rows = y->o_v + up8(y->kv_heads * y->vdim);
    } else {
        y->rank = llmb200_source_dim(&src, "mix.a1", 0);
        if (!y->rank) return -1;
        y->o_k = up8(qk);
        y->o_v = y->o_k + up8(qk);
        y->o_g = y->o_v + up8(hv);
        y->o_f = y->o_g + up8(hv);
        rows = y->o_f + up8(y->rank);
    }
    if (llmb200_new_mat(s, &y->in, rows, D) || llmb200_new_mat(s, &y->o, D, hv) || load_sublayer(m, y, &src, 0, D)) return -1;
    llmb200_load_rows(s, &src, &y->in, "mix.q", qk, D, 0, 1);
    llmb200_load_rows(s, &src, &y->o, "mix.o", D, hv, 0, 1);
    if (y->mixer == MIX_ATTENTION) {
        llmb200_load_rows(s, &src, &y->in, "mix.k", y->kv_heads * y->dim, D, y->o_k, 1);
        llmb200_load_rows(s, &src, &y->in, "mix.v", y->kv_heads * y->vdim, D, y->o_v, 1);
        y->q_gamma = llmb200_load_vec(&src, "mix.q.norm", y->dim, up8(y->dim));
        y->k_gamma = llmb200_load_vec(&src, "mix.k.norm", y->dim, up8(y->dim));
        if (y->temp_every > 0.0 && !(y->q_scale = factor_table(s, m, li))) return -1;
        y->n_split = b200_gqa_splits(s->wtype, y->heads, y->kv_heads, y->dim, y->vdim, s->max_seq);
    } else {
        llmb200_load_rows(s, &src, &y->in, "mix.k", qk, D, y->o_k, 1);
        llmb200_load_rows(s, &src, &y->in, "mix.v", hv, D, y->o_v, 1);
        llmb200_load_rows(s, &src, &y->in, "mix.g", hv, D, y->o_g, 1);
        llmb200_load_rows(s, &src, &y->in, "mix.a1", y->rank, D, y->o_f, 1);
        y->a2 = llmb200_load_table(&src, "mix.a2", qk, y->rank, (y->rank + 3) & ~3);
        y->a2_bias = llmb200_load_vec(&src, "mix.a2.b", qk, qk);
        y->mix_gamma = llmb200_load_vec(&src, "mix.norm", y->vdim, up8(y->vdim));
    }
    if (y->ff) {
        if (llmb200_new_mat(s, &y->up, y->ff, D) || llmb200_new_mat(s, &y->down, D, y->ff) || load_sublayer(m, y, &src, 1, D)) return -1;
        llmb200_load_rows(s, &src, &y->up, "mlp.up", y->ff, D, 0, 1);
        llmb200_load_rows(s, &src, &y->down, "mlp.down", D, y->ff, 0, 1);
    }
    return src.failed ? -1 : 0;
}

/* Cache or state of a run, and its connections: the mix and spread of each sublayer with the take of the one after it
 * (after the last one every stream counts once: the final sum). */
static int make_run(InferenceState *s, Hybrid *m, int r)
{
    Run *run = &m->runs[r];
    const HLayer *y = &m->layers[run->layer], *next = r + 1 < s->L ? &m->layers[m->runs[r + 1].layer] : NULL;
    const int n = m->n_streams;
    if (y->mixer == MIX_ATTENTION) {
        run->k_cache = llmb200_dev_zero((size_t)y->kv_heads * s->max_seq * up8(y->dim) * m->es);
        run->v_cache = llmb200_dev_zero((size_t)y->kv_heads * s->max_seq * up8(y->vdim) * m->es);
        if (!run->k_cache || !run->v_cache) return -1;
    } else {
        run->state = llmb200_dev_zero((size_t)STATE_SLOTS * y->heads * y->dim * up8(y->vdim) * 4);
        if (!run->state) return -1;
    }
    for (int q = 0; q < (y->ff ? 2 : 1); ++q) {
        float c[B200_MAX_STREAMS * (B200_MAX_STREAMS + 2)];
        const float *take = q == 0 && y->ff ? y->take[1] : next ? next->take[0] : NULL;
        memcpy(c, y->mix[q], (size_t)n * n * 4);
        memcpy(c + n * n, y->spread[q], (size_t)n * 4);
        for (int t = 0; t < n; ++t) c[n * n + n + t] = take ? take[t] : 1.0f;
        if (!(run->connect[q] = llmb200_upload_f32(c, (size_t)n * (n + 2)))) return -1;
    }
    const PackedMat *w[] = { &y->in, &y->o, &y->up, &y->down };
    for (int i = 0; i < 4; ++i) s->weight_bytes += (unsigned long long)w[i]->stride * w[i]->rows;
    return 0;
}

static int enqueue_token(InferenceState *s, int with_lm, int pdl);
static int forward_rows(InferenceState *s, const uint32_t *tokens, int n, const int *want, int n_want, float *logits);
static void free_model(InferenceState *s);
static const ModelOps zidepel_ops = { .enqueue_token = enqueue_token, .forward_rows = forward_rows, .free_model = free_model };

InferenceState *llmb200_create_zidepel(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype)
{
    Hybrid *m = calloc(1, sizeof(*m));
    InferenceState *s = m ? llmb200_dir_state(&zidepel_ops, MODEL_ZIDEPEL, m, max_seq_len, wtype) : NULL;
    if (!s) return NULL;
    if (parse(s, m, config) != 0) goto fail;
    m->es = wtype == B200_WT_F32 ? 4 : 2;
    m->Dp = up8(s->D);
    s->V_l = s->V;
    const int n = m->n_streams;
    size_t proj = 0, attn = 0, act = 8, part = 0, tickets = 1;
    for (int i = 0; i < m->n_layers; ++i) {
        if (load_layer(s, m, i, tensors) != 0) { fprintf(stderr, "[FastGen] loading layer %d failed\n", i); goto fail; }
        const HLayer *y = &m->layers[i];
        proj = smax(proj, y->in.rows);
        attn = smax(attn, y->o.cols);
        act = smax(act, y->up.rows);
        if (y->mixer == MIX_ATTENTION) {
            part = smax(part, (size_t)y->heads * y->n_split * (up8(y->vdim) + 8));
            tickets = smax(tickets, (size_t)y->kv_heads * y->heads);
        }
    }
    for (int r = 0; r < s->L; ++r)
        if (make_run(s, m, r) != 0) { fprintf(stderr, "[FastGen] no memory for the cache of layer run %d\n", r); goto fail; }
    TensorSource src = { tensors, -1, 0 };
    if (llmb200_new_mat(s, &m->head, s->V, s->D) != 0) goto fail;
    llmb200_load_rows(s, &src, &m->head, "head", s->V, s->D, 0, 1);
    s->weight_bytes += (unsigned long long)m->head.stride * s->V;
    s->g_final = llmb200_load_vec(&src, "final.norm", s->D, m->Dp);
    m->final_b = llmb200_load_vec(&src, "final.norm.b", s->D, m->Dp);
    m->emb_w = llmb200_load_vec(&src, "embed.norm", s->D, m->Dp);
    m->emb_b = llmb200_load_vec(&src, "embed.norm.b", s->D, m->Dp);
    s->emb = llmb200_load_table(&src, "embed", s->V, s->D, m->Dp);
    m->pos = llmb200_load_table(&src, "pos", m->max_positions, s->D, m->Dp);
    float take = 0.0f;                       /* all streams are x_0 at the start */
    for (int t = 0; t < n; ++t) take += m->layers[m->runs[0].layer].take[0][t];
    m->first_take = llmb200_upload_f32(&take, 1);
    if (src.failed || !m->first_take) goto fail;

    m->proj = llmb200_dev_zero(proj * 4); m->attn = llmb200_dev_zero(attn * 4); m->act = llmb200_dev_zero(act * 4);
    m->part = llmb200_dev_zero(part * 4); m->tickets = (unsigned *)llmb200_dev_zero(tickets * 4);
    m->x0 = llmb200_dev_zero((size_t)m->Dp * 4); m->u = llmb200_dev_zero((size_t)m->Dp * 4);
    for (int i = 0; i < 2; ++i) m->streams[i] = llmb200_dev_zero((size_t)n * m->Dp * 4);
    if (!m->proj || !m->attn || !m->act || !m->part || !m->tickets || !m->x0 || !m->u || !m->streams[0] || !m->streams[1]) goto fail;
    if (llmb200_engine_common(s) != 0 || cudaStreamSynchronize(g_rt.stream) != cudaSuccess) goto fail;
    s->finished = 1;
    return s;
fail:
    inference_state_free(s);
    return NULL;
}

static void free_model(InferenceState *s)
{
    Hybrid *m = s->model;
    if (!m) return;
    for (int i = 0; m->layers && i < m->n_layers; ++i) {
        HLayer *y = &m->layers[i];
        void *b[] = { y->in.w, y->o.w, y->up.w, y->down.w, y->norm_w[0], y->norm_w[1], y->norm_b[0], y->norm_b[1], y->q_gamma, y->k_gamma,
                      y->a2, y->a2_bias, y->mix_gamma };
        for (size_t k = 0; k < sizeof(b) / sizeof(b[0]); ++k) cudaFree(b[k]);
        for (int q = 0; q < 2; ++q) { free(y->take[q]); free(y->spread[q]); free(y->mix[q]); }
    }
    for (int r = 0; m->runs && r < s->L; ++r) {
        Run *run = &m->runs[r];
        void *b[] = { run->k_cache, run->v_cache, run->state, run->connect[0], run->connect[1] };
        for (size_t k = 0; k < sizeof(b) / sizeof(b[0]); ++k) cudaFree(b[k]);
    }
    for (int i = 0; i < m->n_tables; ++i) cudaFree(m->tables[i]);
    void *b[] = { m->head.w, m->pos, m->emb_w, m->emb_b, m->final_b, m->first_take, m->proj, m->attn, m->act, m->part, m->tickets, m->x0,
                  m->streams[0], m->streams[1], m->u, m->r_proj, m->r_x0, m->r_streams[0], m->r_streams[1], m->r_u, m->r_y, m->r_qd, m->r_kd,
                  m->r_decay, m->r_values, m->r_scores, m->r_chunk, m->r_o, m->r_h, m->r_q, m->r_attn, m->r_act };
    for (size_t k = 0; k < sizeof(b) / sizeof(b[0]); ++k) cudaFree(b[k]);
    llmb200_row_path_free(&m->rows);
    free(m->layers);
    free(m->runs);
    free(m->tables);
    free(m);
    s->model = NULL;
}

static void gqa_args(const InferenceState *s, const Hybrid *m, const HLayer *y, const Run *run, const float *proj, b200_gqa_args *a)
{
    memset(a, 0, sizeof(*a));
    a->wtype = s->wtype;
    a->heads = y->heads; a->kv_heads = y->kv_heads; a->dim = y->dim; a->vdim = y->vdim; a->max_seq = s->max_seq;
    a->scale = y->scale; a->softcap = y->softcap; a->eps = m->eps;
    a->d_q = proj; a->d_k = proj + y->o_k; a->d_v = proj + y->o_v;
    a->d_q_gamma = y->q_gamma; a->d_k_gamma = y->k_gamma; a->d_q_scale = y->q_scale;
    a->d_k_cache = run->k_cache; a->d_v_cache = run->v_cache;
}

static void gla_args(const InferenceState *s, const Hybrid *m, const HLayer *y, const Run *run, const float *proj, b200_gla_args *a)
{
    memset(a, 0, sizeof(*a));
    a->wtype = s->wtype;
    a->heads = y->heads; a->dim = y->dim; a->vdim = y->vdim; a->rank = y->rank; a->n_slots = STATE_SLOTS;
    a->tau = y->tau; a->q_scale = (float)(1.0 / sqrt((double)y->dim)); a->eps = m->eps;
    a->d_q = proj; a->d_k = proj + y->o_k; a->d_v = proj + y->o_v; a->d_gate = proj + y->o_g; a->d_f = proj + y->o_f;
    a->d_a2 = y->a2; a->d_a2_bias = y->a2_bias; a->d_norm_gamma = y->mix_gamma;
    a->d_state = run->state;
}

/* ------------------------------------------------------------ one token */

typedef struct { const float *in; long long stride; int to; } Streams;       /* where the old ones are, which buffer is next */

/* The product that reads what the streams hand over: layer norm q of layer y in its input assembly. */
static void reader(InferenceState *s, const Hybrid *m, b200_matvec_args *a, const PackedMat *w, int rows, const float *gamma, const float *beta, int pdl)
{
    llmb200_matvec_base(s, a, w, m->eps, pdl);
    a->rows = rows;
    a->norm_dim = s->D;
    a->in_mode = B200_IN_VEC; a->d_in_vec = m->u;
    a->d_norm_gamma = gamma; a->d_norm_beta = beta;
    a->out_mode = B200_OUT_STORE; a->n_out = 1;
}

/* The product whose result joins the streams. */
static int join(InferenceState *s, const Hybrid *m, const PackedMat *w, const float *in, const float *connect, Streams *x, int last, int kind, int pdl)
{
    b200_matvec_args a;
    llmb200_matvec_base(s, &a, w, m->eps, pdl);
    a.rows = s->D;
    a.in_mode = B200_IN_VEC; a.d_in_vec = in;
    a.out_mode = B200_OUT_STREAMS; a.d_out[0] = m->u; a.n_out = 1;
    a.d_streams_in = x->in; a.streams_in_stride = x->stride;
    a.d_streams_out = m->streams[x->to]; a.streams_out_stride = m->Dp;
    a.d_connect = connect; a.n_streams = m->n_streams;
    x->in = m->streams[x->to]; x->stride = m->Dp; x->to ^= 1;
    if (last) { a.d_ticket = s->mv_ticket; a.advance_pos = 1; a.advance_epoch = 1; }
    llmb200_prof_mark(s, kind);
    if (llmb200_want_kind(s, kind, &a)) K_TRY(b200_matvec(&a, g_rt.stream), return -1);
    llmb200_prof_mark(s, -1);
    return 0;
}

static int enqueue_token(InferenceState *s, int with_lm, int pdl)
{
    const Hybrid *m = s->model;
    void *st = g_rt.stream;
    Streams x = { m->x0, 0, 0 };
    b200_matvec_args a;
    for (int r = 0; r < s->L; ++r) {
        const Run *run = &m->runs[r];
        const HLayer *y = &m->layers[run->layer];
        const int end = !with_lm && r == s->L - 1;
        /* --- everything the mixer takes from this input --- */
        reader(s, m, &a, &y->in, y->in.rows, y->norm_w[0], y->norm_b[0], pdl);
        if (r == 0) {
            a.in_mode = B200_IN_EMBED; a.d_in_vec = NULL;
            a.d_emb = s->emb; a.d_tokens = s->d_tokens; a.emb_scale = 1.0f; a.emb_rows = s->V;
            a.d_emb_pos = m->pos; a.emb_pos_rows = m->max_positions;
            a.d_slot_norm_gamma = m->emb_w; a.d_slot_norm_beta = m->emb_b;
            a.d_resid_out = m->x0; a.d_mix_coef = m->first_take;
        }
        a.d_out[0] = m->proj;
        llmb200_prof_mark(s, K_QKV);
        if (llmb200_want_kind(s, K_QKV, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
        /* --- mixer --- */
        llmb200_prof_mark(s, K_ATTN);
        if (llmb200_want_kind(s, K_ATTN, NULL)) {
            if (y->mixer == MIX_ATTENTION) {
                b200_gqa_args at;
                gqa_args(s, m, y, run, m->proj, &at);
                at.d_part = m->part; at.d_tickets = m->tickets; at.d_out = m->attn; at.d_pos = s->d_pos;
                at.n_split = y->n_split; at.use_pdl = pdl;
                K_TRY(b200_gqa_decode(&at, st), return -1);
            } else {
                b200_gla_args at;
                gla_args(s, m, y, run, m->proj, &at);
                at.d_out = m->attn; at.d_pos = s->d_pos; at.use_pdl = pdl;
                K_TRY(b200_gla_decode(&at, st), return -1);
            }
        }
        llmb200_prof_mark(s, -1);
        if (join(s, m, &y->o, m->attn, run->connect[0], &x, end && !y->ff, K_O, pdl) != 0) return -1;
        if (!y->ff) continue;
        /* --- feed-forward --- */
        reader(s, m, &a, &y->up, y->up.rows, y->norm_w[1], y->norm_b[1], pdl);
        a.act = B200_ACT_RELU2; a.d_out[0] = m->act;
        llmb200_prof_mark(s, K_GATEUP);
        if (llmb200_want_kind(s, K_GATEUP, &a)) K_TRY(b200_matvec(&a, st), return -1);
        llmb200_prof_mark(s, -1);
        if (join(s, m, &y->down, m->act, run->connect[1], &x, end, K_DOWN, pdl) != 0) return -1;
    }
    if (!with_lm) return 0;
    reader(s, m, &a, &m->head, s->V, s->g_final, m->final_b, pdl);
    a.d_out[0] = (float *)(s->comm + s->off_logits);
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

static int rows_ready(InferenceState *s, Hybrid *m)
{
    if (m->rows.chunk) return 0;
    const size_t M = llmb200_row_chunk(s), Dp = m->Dp, n = m->n_streams, es = m->es, nc = (M + CHUNK - 1) / CHUNK;
    size_t proj = 0, q = 0, attn = 0, act = 0, qd = 0, values = 0, decay = 0, scores = 0, chunk = 0, o = 0;
    for (int i = 0; i < m->n_layers; ++i) {
        const HLayer *y = &m->layers[i];
        const size_t wide = (size_t)y->heads * up8(y->dim);
        proj = smax(proj, y->in.rows);
        attn = smax(attn, y->o.cols);
        act = smax(act, y->up.rows);
        if (y->mixer == MIX_ATTENTION) q = smax(q, wide);
        else {
            decay = smax(decay, wide);
            qd = smax(qd, (size_t)3 * CHUNK * y->heads * ((y->dim + 15) & ~15));
            values = smax(values, (size_t)3 * CHUNK * y->heads * up8(y->vdim));
            scores = smax(scores, (size_t)3 * y->heads * CHUNK * CHUNK);
            chunk = smax(chunk, (size_t)3 * y->heads * y->dim * up8(y->vdim));
            if (y->vdim > 128) o = smax(o, (size_t)y->heads * y->vdim);
        }
    }
    m->r_proj = llmb200_dev_zero(M * proj * 4); m->r_x0 = llmb200_dev_zero(M * Dp * 4); m->r_u = llmb200_dev_zero(M * Dp * 4);
    for (int i = 0; i < 2; ++i) m->r_streams[i] = llmb200_dev_zero(n * M * Dp * 4);
    m->r_y = llmb200_dev_zero(M * smax(64, Dp) * 4); m->r_h = llmb200_dev_zero(M * Dp * es);
    m->r_q = llmb200_dev_zero(M * q * es); m->r_attn = llmb200_dev_zero(M * attn * es); m->r_act = llmb200_dev_zero(M * act * es);
    m->r_qd = llmb200_dev_zero(nc * qd * 2); m->r_kd = llmb200_dev_zero(nc * qd * 2); m->r_values = llmb200_dev_zero(nc * values * 2);
    m->r_scores = llmb200_dev_zero(nc * scores * 2); m->r_chunk = llmb200_dev_zero(nc * chunk * 2); m->r_decay = llmb200_dev_zero(nc * decay * 4);
    m->r_o = llmb200_dev_zero(M * o * 4);
    if (!m->r_proj || !m->r_x0 || !m->r_u || !m->r_streams[0] || !m->r_streams[1] || !m->r_y || !m->r_h || !m->r_q || !m->r_attn || !m->r_act ||
        !m->r_qd || !m->r_kd || !m->r_values || !m->r_decay || !m->r_scores || !m->r_chunk || !m->r_o)
        return -1;
    return llmb200_row_path_ready(s, &m->rows, &m->head, m->Dp, (int)M);
}

static int mix_rows(InferenceState *s, Hybrid *m, const HLayer *y, const Run *run, int pos0, int M)
{
    if (y->mixer == MIX_ATTENTION) {
        b200_gqa_args at;
        gqa_args(s, m, y, run, m->r_proj, &at);
        at.n_rows = M; at.pos0 = pos0; at.proj_ld = y->in.rows;
        at.d_q_rows = m->r_q; at.d_out_rows = m->r_attn; at.out_ld = y->o.cols;
        K_TRY(b200_gqa_rows_prep(&at, g_rt.stream), return -1);
        K_TRY(b200_gqa_rows_attend(&at, g_rt.stream), return -1);
        return 0;
    }
    b200_gla_args at;
    gla_args(s, m, y, run, m->r_proj, &at);
    at.n_rows = M; at.pos0 = pos0; at.proj_ld = y->in.rows;
    at.d_qd = m->r_qd; at.d_kd = m->r_kd; at.d_values = m->r_values; at.d_decay = m->r_decay; at.d_scores = m->r_scores; at.d_chunk_state = m->r_chunk; at.d_o = m->r_o;
    at.d_out_rows = m->r_attn; at.out_ld = y->o.cols;
    K_TRY(b200_gla_rows(&at, g_rt.stream), return -1);
    return 0;
}

/* M tokens from position pos0 on, whose ids are in d_tokens; the sum of the streams is left in r_u. */
static int pass_rows(InferenceState *s, int pos0, int M)
{
    Hybrid *m = s->model;
    const int Dp = m->Dp;
    const long long plane = (long long)m->rows.chunk * Dp;
    const HLayer *first = &m->layers[m->runs[0].layer];
    b200_rows_start_args b;
    memset(&b, 0, sizeof(b));
    b.emb = s->emb; b.emb_pos = m->pos; b.tokens = (const uint32_t *)s->d_tokens + pos0; b.vocab = s->V; b.pos_rows = m->max_positions; b.pos0 = pos0;
    b.emb_gamma = m->emb_w; b.emb_beta = m->emb_b; b.take = m->first_take; b.gamma = first->norm_w[0]; b.beta = first->norm_b[0]; b.eps = m->eps;
    b.rows = M; b.dim = s->D; b.ld = Dp; b.wtype = s->wtype;
    b.x = m->r_x0; b.out = m->r_h;
    K_TRY(b200_rows_start(&b, g_rt.stream), return -1);

    b200_rows_streams_args j;
    memset(&j, 0, sizeof(j));
    j.n_streams = m->n_streams; j.eps = m->eps; j.rows = M; j.dim = s->D; j.ld = Dp; j.wtype = s->wtype;
    j.streams_in = m->r_x0;
    j.y = m->r_y;
    int to = 0;
    for (int r = 0; r < s->L; ++r) {
        const Run *run = &m->runs[r];
        const HLayer *y = &m->layers[run->layer];
        for (int q = 0; q < (y->ff ? 2 : 1); ++q) {
            const PackedMat *w = q ? &y->down : &y->o;
            if (q == 0) {
                if (llmb200_rows_product(s, m->r_h, Dp, &y->in, M, m->r_proj, y->in.rows, NULL, 0) || mix_rows(s, m, y, run, pos0, M) ||
                    llmb200_rows_product(s, m->r_attn, y->o.cols, w, M, m->r_y, w->rows, NULL, 0))
                    return -1;
            } else if (llmb200_rows_product(s, m->r_h, Dp, &y->up, M, NULL, y->up.rows, m->r_act, 1) ||
                       llmb200_rows_product(s, m->r_act, y->up.rows, w, M, m->r_y, w->rows, NULL, 0))
                return -1;
            /* join the result, and the next reader's norm */
            const int more = q == 0 && y->ff, end = !more && r == s->L - 1;
            const HLayer *next = more ? y : end ? NULL : &m->layers[m->runs[r + 1].layer];
            j.y_ld = w->rows;
            j.connect = run->connect[q];
            j.gamma = next ? next->norm_w[more] : NULL; j.beta = next ? next->norm_b[more] : NULL;
            j.streams_out = end ? NULL : m->r_streams[to]; j.streams_out_stride = plane;
            j.u_out = end ? m->r_u : NULL;
            j.out = end ? NULL : m->r_h;
            K_TRY(b200_rows_streams(&j, g_rt.stream), return -1);
            j.streams_in = m->r_streams[to]; j.streams_in_stride = plane;
            to ^= 1;
        }
    }
    return 0;
}

static int last_rows(InferenceState *s, const int *index, int n, void *out)
{
    const Hybrid *m = s->model;
    K_TRY(b200_rows_layer_norm(m->r_u, index, n, s->D, m->Dp, m->eps, s->g_final, m->final_b, s->wtype, out, g_rt.stream), return -1);
    return 0;
}

static int forward_rows(InferenceState *s, const uint32_t *tokens, int n, const int *want, int n_want, float *logits)
{
    Hybrid *m = s->model;
    if (rows_ready(s, m) != 0) { fprintf(stderr, "[FastGen] no memory for the row path\n"); return -1; }
    return llmb200_row_path_run(s, &m->rows, pass_rows, last_rows, 0.0f, tokens, n, want, n_want, logits);
}
