/* Constructors of the model types that are built from a folder (internal). */
#ifndef LLMB200_MODEL_DIR_H
#define LLMB200_MODEL_DIR_H

#include "engine.h"
#include "json.h"
#include "tensor_file.h"

InferenceState *llmb200_create_morilorn(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype);

#endif
