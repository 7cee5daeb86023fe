/* What the model types built from a folder share (see model_dir.h). */
#include "model_dir.h"
#include "../../include/llmb200_train_kernels.h"

#include <stdlib.h>
#include <string.h>

enum { ROW_CHUNK = 2048, WANT_CHUNK = 256 };

InferenceState *llmb200_dir_state(const ModelOps *ops, ModelType mt, void *model, int max_seq_len, int wtype)
{
    if (fast_metal_init() != 0) { fprintf(stderr, "[FastGen] CUDA init failed\n"); free(model); return NULL; }
    InferenceState *s = calloc(1, sizeof(*s));
    if (!s) { fast_metal_shutdown(); free(model); return NULL; }
    s->ops = ops;
    s->model = model;
    s->mt = mt;
    s->wtype = wtype;
    s->max_seq = max_seq_len;
    llmb200_engine_tp(&s->tp_rank, &s->tp_size);
    const int world = s->tp_size;
    s->tp_rank = 0;
    s->tp_size = 1;
    if (world != 1) fprintf(stderr, "[FastGen] this model type runs on one GPU\n");
    if (world != 1 || cudaDeviceGetAttribute(&s->n_sm, cudaDevAttrMultiProcessorCount, g_rt.device) != cudaSuccess || s->n_sm <= 0) {
        inference_state_free(s);
        return NULL;
    }
    return s;
}

int llmb200_bad_config(const char *where, const char *what)
{
    fprintf(stderr, "[FastGen] config.json: %s: %s\n", where, what);
    return -1;
}

/* ------------------------------------------------------------ loading */

int llmb200_new_mat(InferenceState *s, PackedMat *m, int rows, int cols)
{
    m->rows = rows > 64 ? llmb200_up8(rows) : 64;
    m->cols = llmb200_up8(cols);
    m->stride = (long long)b200_packed_row_stride(s->wtype, m->cols);
    m->w = llmb200_dev_zero((size_t)m->stride * m->rows);
    return m->w ? 0 : -1;
}

int llmb200_put_rows(InferenceState *s, PackedMat *m, const float *src, int rows, int cols, int row0, int step)
{
    return llmb200_upload_packed(s->wtype, src, cols, rows, 0, cols, m->w, m->stride, row0, step);
}

static void full_name(const TensorSource *src, const char *name, char *out, size_t cap)
{
    if (src->layer >= 0) snprintf(out, cap, "l%d.%s", src->layer, name);
    else snprintf(out, cap, "%s", name);
}

float *llmb200_source_tensor(TensorSource *src, const char *name, long long d0, long long d1)
{
    char full[128];
    full_name(src, name, full, sizeof(full));
    float *t = llmb200_tensor_f32(src->file, full, d0, d1);
    if (!t) src->failed = 1;
    return t;
}

int llmb200_source_dim(TensorSource *src, const char *name, int axis)
{
    char full[128];
    full_name(src, name, full, sizeof(full));
    const long long n = llmb200_tensor_dim(src->file, full, axis);
    if (n < 1 || n > 0x7fffffff) { fprintf(stderr, "[llmb200] tensor %s is missing or has another rank\n", full); src->failed = 1; return 0; }
    return (int)n;
}

void llmb200_load_rows(InferenceState *s, TensorSource *src, PackedMat *m, const char *name, int rows, int cols, int row0, int step)
{
    float *t = llmb200_source_tensor(src, name, rows, cols);
    if (t && llmb200_put_rows(s, m, t, rows, cols, row0, step) != 0) src->failed = 1;
    free(t);
}

float *llmb200_load_vec(TensorSource *src, const char *name, int n, int padded)
{
    float *t = llmb200_source_tensor(src, name, n, 0), *d = t ? llmb200_dev_zero((size_t)padded * 4) : NULL;
    if (!d || llmb200_upload_f32_into(d, t, (size_t)n) != 0) src->failed = 1;
    free(t);
    return d;
}

float *llmb200_load_table(TensorSource *src, const char *name, int rows, int cols, int ld)
{
    float *t = llmb200_source_tensor(src, name, rows, cols), *d = t ? llmb200_dev_zero((size_t)rows * ld * 4) : NULL;
    if (!d || llmb200_upload_packed(B200_WT_F32, t, cols, rows, 0, cols, d, (long long)ld * 4, 0, 1) != 0) src->failed = 1;
    free(t);
    return d;
}

/* ------------------------------------------------------------ rows */

int llmb200_rows_product(InferenceState *s, const void *A, long long lda, const PackedMat *w, int M, float *C, long long ldc, void *Ch, int relu2)
{
    const int f32 = s->wtype == B200_WT_F32;
    b200_gemm_args g;
    memset(&g, 0, sizeof(g));
    g.A = A; g.a_row = lda; g.a_col = 1;
    g.B = w->w; g.b_row = 1; g.b_col = w->stride / (f32 ? 4 : 2);
    g.ldc = ldc; g.M = M; g.N = w->rows; g.K = w->cols; g.alpha = 1.0f;
    g.d_err = (unsigned *)s->d_err;
    g.relu2 = relu2;
    if (Ch && !f32) { g.Ch = Ch; g.ldch = ldc; }
    else g.C = Ch ? Ch : C;
    const int rc = f32 ? b200_gemm_f32(&g, g_rt.stream) : b200_gemm_bf16(&g, g_rt.stream);
    if (rc) fprintf(stderr, "[FastGen] row product %d x %d x %d failed: code %d\n", M, w->rows, w->cols, rc);
    return rc;
}

int llmb200_row_chunk(const InferenceState *s) { return s->max_seq < ROW_CHUNK ? s->max_seq : ROW_CHUNK; }

int llmb200_row_path_ready(InferenceState *s, RowPath *r, const PackedMat *head, int ld, int chunk)
{
    const size_t wc = s->max_seq < WANT_CHUNK ? s->max_seq : WANT_CHUNK;
    r->head = head;
    r->ld = ld;
    r->want_chunk = (int)wc;
    r->last = llmb200_dev_zero(wc * ld * (s->wtype == B200_WT_F32 ? 4 : 2));
    r->logits = llmb200_dev_zero(wc * head->rows * 4);
    r->d_want = (int *)llmb200_dev_zero(wc * 4);
    if (!r->last || !r->logits || !r->d_want) return -1;
    CU_TRY(cudaMallocHost((void **)&r->h_want, wc * 4), return -1);
    r->chunk = chunk;
    return 0;
}

void llmb200_row_path_free(RowPath *r)
{
    cudaFree(r->last);
    cudaFree(r->logits);
    cudaFree(r->d_want);
    if (r->h_want) cudaFreeHost(r->h_want);
}

int llmb200_row_path_run(InferenceState *s, RowPath *r, int (*pass)(InferenceState *s, int pos0, int M),
                         int (*last)(InferenceState *s, const int *index, int n, void *out), float softcap,
                         const uint32_t *tokens, int n, const int *want, int n_want, float *logits)
{
    int w = 0;
    for (int c0 = 0; c0 < n; c0 += r->chunk) {
        const int M = n - c0 < r->chunk ? n - c0 : r->chunk, pos0 = s->cur_len + c0;
        if (llmb200_set_control(s, pos0, s->max_seq + 2, tokens + c0, pos0, M) != 0) return -1;
        if (pass(s, pos0, M) != 0) return -1;
        while (w < n_want && want[w] < c0 + M) {
            int k = 0;
            CU_TRY(cudaStreamSynchronize(g_rt.stream), return -1);           /* h_want may still be in flight */
            while (k < r->want_chunk && w + k < n_want && want[w + k] < c0 + M) { r->h_want[k] = want[w + k] - c0; ++k; }
            CU_TRY(cudaMemcpyAsync(r->d_want, r->h_want, (size_t)k * 4, cudaMemcpyHostToDevice, g_rt.stream), return -1);
            if (last(s, r->d_want, k, r->last) != 0) return -1;
            if (llmb200_rows_product(s, r->last, r->ld, r->head, k, r->logits, r->head->rows, NULL, 0)) return -1;
            if (softcap > 0.0f) K_TRY(b200_rows_softcap(r->logits, k, s->V, r->head->rows, softcap, g_rt.stream), return -1);
            CU_TRY(cudaMemcpy2DAsync(logits + (size_t)w * s->V, (size_t)s->V * 4, r->logits, (size_t)r->head->rows * 4, (size_t)s->V * 4, (size_t)k,
                                     cudaMemcpyDeviceToHost, g_rt.stream), return -1);
            w += k;
        }
    }
    CU_TRY(cudaStreamSynchronize(g_rt.stream), return -1);
    return 0;
}
