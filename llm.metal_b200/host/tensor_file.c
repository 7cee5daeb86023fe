/* safetensors reader (see tensor_file.h). */
#include "tensor_file.h"
#include "json.h"

#include <fcntl.h>
#include <stdint.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

struct llmb200_tensor_file {
    unsigned char *map;
    size_t size, data;           /* mapped bytes; where the data section starts */
    json *header;
};

llmb200_tensor_file *llmb200_tensor_file_open(const char *path)
{
    llmb200_tensor_file *f = calloc(1, sizeof(*f));
    const int fd = f ? open(path, O_RDONLY) : -1;
    struct stat st;
    if (fd < 0 || fstat(fd, &st) != 0 || st.st_size < 8) {
        fprintf(stderr, "[llmb200] cannot read %s\n", path);
        if (fd >= 0) close(fd);
        free(f);
        return NULL;
    }
    f->size = (size_t)st.st_size;
    f->map = mmap(NULL, f->size, PROT_READ, MAP_PRIVATE, fd, 0);
    close(fd);
    if (f->map == MAP_FAILED) { fprintf(stderr, "[llmb200] cannot map %s\n", path); free(f); return NULL; }
    uint64_t n = 0;
    for (int i = 0; i < 8; ++i) n |= (uint64_t)f->map[i] << (8 * i);
    if (n <= f->size - 8) {
        f->header = json_parse((const char *)f->map + 8, (size_t)n, NULL);
        f->data = 8 + (size_t)n;
    }
    if (!f->header || f->header->type != JSON_OBJECT) {
        fprintf(stderr, "[llmb200] %s is not a safetensors file\n", path);
        llmb200_tensor_file_close(f);
        return NULL;
    }
    return f;
}

void llmb200_tensor_file_close(llmb200_tensor_file *f)
{
    if (!f) return;
    if (f->map && f->map != MAP_FAILED) munmap(f->map, f->size);
    json_free(f->header);
    free(f);
}

static float half_to_f32(uint16_t h)
{
    const uint32_t sign = (uint32_t)(h >> 15) << 31, ex = (h >> 10) & 31, man = h & 1023;
    uint32_t b;
    if (ex == 31) b = sign | 0x7f800000u | (man << 13);
    else if (ex) b = sign | ((ex + 112) << 23) | (man << 13);
    else {
        const float v = (float)man * 5.9604644775390625e-08f;          /* subnormal: man * 2^-24 */
        memcpy(&b, &v, 4);
        b |= sign;
    }
    float r;
    memcpy(&r, &b, 4);
    return r;
}

float *llmb200_tensor_f32(const llmb200_tensor_file *f, const char *name, long long d0, long long d1)
{
    const json *t = json_get(f->header, name);
    const json *shape = json_get(t, "shape"), *off = json_get(t, "data_offsets");
    const char *dtype = json_string(t, "dtype");
    const int rank = d1 > 0 ? 2 : 1;
    if (!t || !dtype || !shape || shape->type != JSON_ARRAY || !off || off->type != JSON_ARRAY || off->n != 2) {
        fprintf(stderr, "[llmb200] tensor %s is missing\n", name);
        return NULL;
    }
    if (shape->n != rank || shape->child->number != (double)d0 || (rank == 2 && shape->child->next->number != (double)d1)) {
        fprintf(stderr, "[llmb200] tensor %s has another shape than [%lld%s%.0lld]\n", name, d0, rank == 2 ? ", " : "", d1);
        return NULL;
    }
    const int es = !strcmp(dtype, "BF16") || !strcmp(dtype, "F16") ? 2 : !strcmp(dtype, "F32") ? 4 : 0;
    const size_t n = (size_t)d0 * (size_t)(rank == 2 ? d1 : 1);
    const double a = off->child->number, b = off->child->next->number;
    if (!es || a < 0 || b < a || b - a != (double)n * es || b > (double)(f->size - f->data)) {
        fprintf(stderr, "[llmb200] tensor %s: unsupported type or damaged offsets\n", name);
        return NULL;
    }
    float *out = malloc((n ? n : 1) * sizeof(float));
    if (!out) { fprintf(stderr, "[llmb200] out of memory for tensor %s\n", name); return NULL; }
    const unsigned char *src = f->map + f->data + (size_t)a;
    if (es == 4) memcpy(out, src, n * 4);
    else if (dtype[0] == 'B')
        for (size_t i = 0; i < n; ++i) {
            const uint32_t w = (uint32_t)src[2 * i + 1] << 24 | (uint32_t)src[2 * i] << 16;
            memcpy(out + i, &w, 4);
        }
    else
        for (size_t i = 0; i < n; ++i) out[i] = half_to_f32((uint16_t)(src[2 * i] | src[2 * i + 1] << 8));
    return out;
}

long long llmb200_tensor_dim(const llmb200_tensor_file *f, const char *name, int axis)
{
    const json *shape = json_get(json_get(f->header, name), "shape");
    if (!shape || shape->type != JSON_ARRAY || axis < 0 || axis >= shape->n) return -1;
    const json *d = shape->child;
    while (axis-- > 0) d = d->next;
    return d->type == JSON_NUMBER && d->number >= 0 && d->number < 9e15 ? (long long)d->number : -1;
}
