/* Constructors of the model types that are built from a folder, and what they share: loading into packed matrices,
 * products of the row path, and the loop over a prompt portion (internal). */
#ifndef LLMB200_MODEL_DIR_H
#define LLMB200_MODEL_DIR_H

#include "engine.h"
#include "json.h"
#include "tensor_file.h"

InferenceState *llmb200_create_morilorn(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype);
InferenceState *llmb200_create_zidepel(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype);

static inline int llmb200_up8(int n) { return (n + 7) & ~7; }

/* A zeroed state of the folder's model type on one GPU, the owner of `model` (zeroed heap memory) from here on; NULL with
 * a message, `model` freed, when it cannot be made. */
InferenceState *llmb200_dir_state(const ModelOps *ops, ModelType mt, void *model, int max_seq_len, int wtype);
int llmb200_bad_config(const char *where, const char *what);      /* message on stderr, -1 */

/* Tensors "l<layer>.<name>" of a file, or "<name>" when layer < 0. A failure is remembered in `failed`. */
typedef struct { const llmb200_tensor_file *file; int layer; int failed; } TensorSource;

/* A matrix of rows x up8(cols), zero; at least 64 rows, the narrowest the tensor-core product takes. */
int llmb200_new_mat(InferenceState *s, PackedMat *m, int rows, int cols);
int llmb200_put_rows(InferenceState *s, PackedMat *m, const float *src, int rows, int cols, int row0, int step);
/* A tensor as fp32 on the host (d1 = 0: a vector); the caller frees it. */
float *llmb200_source_tensor(TensorSource *src, const char *name, long long d0, long long d1);
int llmb200_source_dim(TensorSource *src, const char *name, int axis);        /* a dimension of a tensor; 0 when there is none */
void llmb200_load_rows(InferenceState *s, TensorSource *src, PackedMat *m, const char *name, int rows, int cols, int row0, int step);
/* A vector of n elements, zero-padded to `padded` on the device. */
float *llmb200_load_vec(TensorSource *src, const char *name, int n, int padded);
/* An fp32 table on the device, its rows zero-padded to `ld` columns. */
float *llmb200_load_table(TensorSource *src, const char *name, int rows, int cols, int ld);

/* C[M, w->rows] = A[M, K] x w^T; A has the matrices' element type, K columns (padding included) lda apart. Ch: the
 * result in that element type instead of C. relu2 (with Ch): the squared relu of the result. */
int llmb200_rows_product(InferenceState *s, const void *A, long long lda, const PackedMat *w, int M, float *C, long long ldc, void *Ch, int relu2);

/* A prompt portion runs in passes of up to `chunk` tokens; logits are formed for the wanted rows only. */
typedef struct { int chunk, want_chunk, ld; const PackedMat *head; void *last; float *logits; int *d_want, *h_want; } RowPath;
int llmb200_row_chunk(const InferenceState *s);
int llmb200_row_path_ready(InferenceState *s, RowPath *r, const PackedMat *head, int ld, int chunk);
void llmb200_row_path_free(RowPath *r);
/* `pass` runs M tokens from position pos0 on, whose ids are on the device; `last` makes the head's input (final norm) of
 * the n rows index[] of the pass, ld elements apart. */
int llmb200_row_path_run(InferenceState *s, RowPath *r, int (*pass)(InferenceState *s, int pos0, int M),
                         int (*last)(InferenceState *s, const int *index, int n, void *out), float softcap,
                         const uint32_t *tokens, int n, const int *want, int n_want, float *logits);

#endif
