// Row-wise steps of a prompt portion (sm_100a): embedding, grouped RMS norms after a gated, scaled residual sum,
// the depth average over earlier layers' results, GeGLU and the logit cap. One block per row; every sum is formed
// in a fixed order. Results that a tensor-core product reads next are written as bfloat16 too.
#include "stream_core.cuh"
#include "../../include/llmb200_kernels.h"

#include <cuda_bf16.h>

extern unsigned long long g_b200_launches;

namespace {

__global__ void __launch_bounds__(256)
rows_embed_kernel(const float *emb, const uint32_t *tokens, int vocab, int ld, float scale, float *x, __nv_bfloat16 *xh)
{
    const size_t m = blockIdx.x;
    uint32_t t = tokens[m];
    if (t >= (uint32_t)vocab) t = 0;                         // never outside the table
    for (int i = threadIdx.x; i < ld; i += 256) {
        const float v = emb[(size_t)t * ld + i] * scale;
        x[m * ld + i] = v;
        if (xh) xh[m * ld + i] = __float2bfloat16_rn(v);
    }
}

// 1 / rms of each of `groups` equal parts of row[0 .. dim) (shared memory) into inv[groups].
__device__ __forceinline__ void part_scales(const float *row, int dim, int groups, float eps, float *red, float *inv)
{
    const int len = dim / groups;
    for (int g = 0; g < groups; ++g) {
        float ss = 0.0f;
        for (int i = g * len + threadIdx.x; i < (g + 1) * len; i += blockDim.x) ss = fmaf(row[i], row[i], ss);
        ss = block_sum(ss, red);
        if (threadIdx.x == 0) inv[g] = 1.0f / sqrtf(ss / (float)len + eps);
    }
    __syncthreads();
}

__global__ void __launch_bounds__(256) rows_postnorm_kernel(const b200_rows_postnorm_args p)
{
    extern __shared__ float sh[];                            // [dim] row, [groups] scales
    __shared__ float red[33];
    float *row = sh, *inv = sh + p.dim;
    const size_t m = blockIdx.x;
    const float *x = p.x + m * p.ld, *y = p.y + m * p.y_ld, *gate = p.gate + m * p.gate_ld;
    for (int i = threadIdx.x; i < p.dim; i += 256) row[i] = fmaf(p.alpha, x[i], sigmoid_f32(gate[i] + p.gate_bias[i]) * y[i]);
    __syncthreads();
    part_scales(row, p.dim, p.groups, p.eps, red, inv);
    const int len = p.dim / p.groups;
    __nv_bfloat16 *oh = static_cast<__nv_bfloat16 *>(p.out_h);
    const float c_new = p.hist_n > 0 ? p.coef[p.hist_n] : 1.0f;
    for (int i = threadIdx.x; i < p.ld; i += 256) {
        float v = 0.0f;
        if (i < p.dim) {
            v = p.gamma[i] * (row[i] * inv[i / len]);
            if (p.norm_out) p.norm_out[m * p.ld + i] = v;
            if (p.hist_n > 0) {
                float a = 0.0f;
#pragma unroll 8
                for (int j = 0; j < p.hist_n; ++j) a = fmaf(p.coef[j], p.hist[(size_t)j * p.hist_stride + m * p.ld + i], a);
                v = fmaf(c_new, v, a);
            }
        } else if (p.norm_out) p.norm_out[m * p.ld + i] = 0.0f;
        if (p.out != p.norm_out || p.hist_n > 0) p.out[m * p.ld + i] = v;
        if (oh) oh[m * p.ld + i] = __float2bfloat16_rn(v);
    }
}

template <typename T>
__global__ void __launch_bounds__(256)
rows_norm_kernel(const float *x, const int *index, int dim, int ld, int groups, float eps, const float *gamma, T *out)
{
    extern __shared__ float sh[];
    __shared__ float red[33];
    float *row = sh, *inv = sh + dim;
    const size_t m = blockIdx.x, src = index ? (size_t)index[m] : m;
    for (int i = threadIdx.x; i < dim; i += 256) row[i] = x[src * ld + i];
    __syncthreads();
    part_scales(row, dim, groups, eps, red, inv);
    const int len = dim / groups;
    for (int i = threadIdx.x; i < ld; i += 256) out[m * ld + i] = (T)(i < dim ? gamma[i] * (row[i] * inv[i / len]) : 0.0f);
}

template <typename T>
__global__ void __launch_bounds__(256) rows_gelu_mul_kernel(const float *gu, long long ld, int rows, int inter, T *out)
{
    const size_t total = (size_t)rows * inter;
    for (size_t e = (size_t)blockIdx.x * 256 + threadIdx.x; e < total; e += (size_t)gridDim.x * 256) {
        const size_t m = e / inter, i = e % inter;
        const float2 v = *reinterpret_cast<const float2 *>(gu + m * ld + 2 * i);
        out[e] = (T)(act_gelu_tanh(v.x) * v.y);
    }
}

__global__ void __launch_bounds__(256) rows_softcap_kernel(float *x, int rows, int dim, long long ld, float cap)
{
    const size_t total = (size_t)rows * dim;
    for (size_t e = (size_t)blockIdx.x * 256 + threadIdx.x; e < total; e += (size_t)gridDim.x * 256) {
        float *v = x + (e / dim) * ld + e % dim;
        *v = cap * tanhf(*v / cap);
    }
}

unsigned grid_for(size_t total)
{
    const size_t g = (total + 255) / 256;
    return (unsigned)(g < 148 * 16 ? g : 148 * 16);
}

int done() { ++g_b200_launches; return (int)cudaGetLastError(); }

template <typename K>
int row_smem(K kern, size_t smem)
{
    if (smem > 220 * 1024) return B200_E_TOOLARGE;
    return smem > 40 * 1024 ? (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : 0;
}

}  // namespace

extern "C" int b200_rows_embed(const float *emb, const uint32_t *tokens, int rows, int vocab, int ld, float scale,
                               float *x, void *out_h, void *stream)
{
    if (!emb || !tokens || !x || rows <= 0 || vocab <= 0 || ld <= 0) return B200_E_BADARG;
    rows_embed_kernel<<<rows, 256, 0, (cudaStream_t)stream>>>(emb, tokens, vocab, ld, scale, x, static_cast<__nv_bfloat16 *>(out_h));
    return done();
}

extern "C" int b200_rows_postnorm(const b200_rows_postnorm_args *a, void *stream)
{
    if (!a || !a->x || !a->y || !a->gate || !a->gate_bias || !a->gamma || !a->out || a->rows <= 0 || a->dim <= 0 || a->ld < a->dim ||
        a->groups <= 0 || a->dim % a->groups || a->hist_n < 0 || (a->hist_n > 0 && (!a->hist || !a->coef)))
        return B200_E_BADARG;
    const size_t smem = (size_t)(a->dim + a->groups) * 4;
    const int rc = row_smem(rows_postnorm_kernel, smem);
    if (rc) return rc;
    rows_postnorm_kernel<<<a->rows, 256, smem, (cudaStream_t)stream>>>(*a);
    return done();
}

extern "C" int b200_rows_norm(const float *x, const int *index, int rows, int dim, int ld, int groups, float eps,
                              const float *gamma, int wtype, void *out, void *stream)
{
    if (!x || !gamma || !out || rows <= 0 || dim <= 0 || ld < dim || groups <= 0 || dim % groups ||
        (wtype != B200_WT_BF16 && wtype != B200_WT_F32))
        return B200_E_BADARG;
    const size_t smem = (size_t)(dim + groups) * 4;
    cudaStream_t st = (cudaStream_t)stream;
    int rc;
    if (wtype == B200_WT_BF16) {
        if ((rc = row_smem(rows_norm_kernel<__nv_bfloat16>, smem)) != 0) return rc;
        rows_norm_kernel<__nv_bfloat16><<<rows, 256, smem, st>>>(x, index, dim, ld, groups, eps, gamma, static_cast<__nv_bfloat16 *>(out));
    } else {
        if ((rc = row_smem(rows_norm_kernel<float>, smem)) != 0) return rc;
        rows_norm_kernel<float><<<rows, 256, smem, st>>>(x, index, dim, ld, groups, eps, gamma, static_cast<float *>(out));
    }
    return done();
}

extern "C" int b200_rows_gelu_mul(const float *gu, long long gu_ld, int rows, int inter, int wtype, void *out, void *stream)
{
    if (!gu || !out || rows <= 0 || inter <= 0 || gu_ld < 2LL * inter || (gu_ld & 1) || (wtype != B200_WT_BF16 && wtype != B200_WT_F32))
        return B200_E_BADARG;
    const unsigned grid = grid_for((size_t)rows * inter);
    cudaStream_t st = (cudaStream_t)stream;
    if (wtype == B200_WT_BF16) rows_gelu_mul_kernel<<<grid, 256, 0, st>>>(gu, gu_ld, rows, inter, static_cast<__nv_bfloat16 *>(out));
    else rows_gelu_mul_kernel<<<grid, 256, 0, st>>>(gu, gu_ld, rows, inter, static_cast<float *>(out));
    return done();
}

extern "C" int b200_rows_softcap(float *x, int rows, int dim, long long ld, float cap, void *stream)
{
    if (!x || rows <= 0 || dim <= 0 || ld < dim || !(cap > 0.0f)) return B200_E_BADARG;
    rows_softcap_kernel<<<grid_for((size_t)rows * dim), 256, 0, (cudaStream_t)stream>>>(x, rows, dim, ld, cap);
    return done();
}
