/*
 * Models described by a folder: config.json + model.safetensors. config.json's "architecture" selects the
 * model type; every type registers one constructor here.
 */
#include "engine.h"
#include "model_dir.h"

#include <stdlib.h>
#include <string.h>

static const struct {
    const char *architecture;
    InferenceState *(*create)(const json *config, const llmb200_tensor_file *tensors, int max_seq_len, int wtype);
} registry[] = {
    { "Morilorn", llmb200_create_morilorn },
    { "Zidepel", llmb200_create_zidepel },
};

InferenceState *inference_state_create_from_dir(const char *dir, int max_seq_len, int wtype)
{
    if (!dir || max_seq_len <= 0 || (wtype != B200_WT_BF16 && wtype != B200_WT_F32)) {
        fprintf(stderr, "[FastGen] a model folder needs a positive cache length and bfloat16 or fp32 as its type\n");
        return NULL;
    }
    const size_t n = strlen(dir) + 32;
    char *path = malloc(n);
    if (!path) return NULL;
    InferenceState *s = NULL;
    snprintf(path, n, "%s/config.json", dir);
    char *text = llmb200_slurp(path);
    size_t at = 0;
    json *config = text ? json_parse(text, strlen(text), &at) : NULL;
    llmb200_tensor_file *tensors = NULL;
    if (!config) {
        if (text) fprintf(stderr, "[FastGen] %s: not valid JSON (offset %zu)\n", path, at);
        else fprintf(stderr, "[FastGen] cannot read %s\n", path);
        goto out;
    }
    const char *arch = json_string(config, "architecture");
    size_t k = 0;
    while (k < sizeof(registry) / sizeof(registry[0]) && (!arch || strcmp(arch, registry[k].architecture))) ++k;
    if (k == sizeof(registry) / sizeof(registry[0])) {
        fprintf(stderr, "[FastGen] %s: unknown architecture \"%s\"\n", path, arch ? arch : "");
        goto out;
    }
    snprintf(path, n, "%s/model.safetensors", dir);
    tensors = llmb200_tensor_file_open(path);
    if (!tensors) goto out;
    s = registry[k].create(config, tensors, max_seq_len, wtype);
    if (s && json_get(config, "eos_token_id")) inference_state_load_eos(s, dir);
out:
    llmb200_tensor_file_close(tensors);
    json_free(config);
    free(text);
    free(path);
    return s;
}
