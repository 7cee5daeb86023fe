/* Read access to a safetensors file: an 8-byte little-endian length, that many bytes of JSON
 * (name -> dtype, shape, data_offsets), then the data. The file is mapped, not read. */
#ifndef LLMB200_TENSOR_FILE_H
#define LLMB200_TENSOR_FILE_H

#include <stddef.h>

typedef struct llmb200_tensor_file llmb200_tensor_file;

llmb200_tensor_file *llmb200_tensor_file_open(const char *path);   /* NULL with a message on stderr */
void llmb200_tensor_file_close(llmb200_tensor_file *f);
/* A heap copy of a BF16, F16 or F32 tensor as fp32. d1 = 0: a vector of d0 elements, else a [d0, d1] matrix.
 * NULL with a message on stderr when the tensor is missing or has another shape or type. */
float *llmb200_tensor_f32(const llmb200_tensor_file *f, const char *name, long long d0, long long d1);
/* Length of a tensor's axis, -1 when the tensor or the axis does not exist. */
long long llmb200_tensor_dim(const llmb200_tensor_file *f, const char *name, int axis);

#endif
