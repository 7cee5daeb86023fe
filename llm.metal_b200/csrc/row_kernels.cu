// Row-wise steps of a prompt portion (sm_100a): embedding, grouped RMS norms after a gated, scaled residual sum,
// the depth average over earlier layers' results, layer norms, residual streams, GeGLU and the logit cap. One block per row; every sum is formed
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

__device__ __forceinline__ void store4(float *out, const float4 &v) { *reinterpret_cast<float4 *>(out) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *out, const float4 &v)
{
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(out) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}

// Layer norm of row[0 .. dim) (shared memory; this thread wrote quads threadIdx.x + 256 k, `sum` is the sum of what it
// wrote, elements past dim are zeros). Every quad below ld goes through `put` with its normalised value.
template <typename Put>
__device__ __forceinline__ void layer_norm_row(float *row, float sum, int dim, int ld, float eps, const float *gamma, const float *beta,
                                               float *red, Put put)
{
    const float mean = block_sum(sum, red) / (float)dim;
    float ss = 0.0f;
    for (int i = 4 * threadIdx.x; i < ld; i += 1024)
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (i + e < dim) { const float d = row[i + e] - mean; ss = fmaf(d, d, ss); }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)dim + eps);
    for (int i = 4 * threadIdx.x; i < ld; i += 1024) {
        const float4 x = *reinterpret_cast<const float4 *>(row + i), g = *reinterpret_cast<const float4 *>(gamma + i), b = *reinterpret_cast<const float4 *>(beta + i);
        put(i, make_float4(fmaf(g.x, (x.x - mean) * inv, b.x), fmaf(g.y, (x.y - mean) * inv, b.y),
                           fmaf(g.z, (x.z - mean) * inv, b.z), fmaf(g.w, (x.w - mean) * inv, b.w)));
    }
}

template <typename T>
__global__ void __launch_bounds__(256) rows_streams_kernel(const b200_rows_streams_args p)
{
    extern __shared__ __align__(16) float row[];             // [ld]
    __shared__ float red[33], conn[B200_MAX_STREAMS * (B200_MAX_STREAMS + 2)];
    const int n = p.n_streams;
    if ((int)threadIdx.x < n * (n + 2)) conn[threadIdx.x] = p.connect[threadIdx.x];
    __syncthreads();
    const size_t m = blockIdx.x;
    const float *xin = p.streams_in + m * p.ld, *y = p.y + m * p.y_ld;
    float sum = 0.0f;
    for (int i = 4 * threadIdx.x; i < p.ld; i += 1024) {
        float4 x[B200_MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < B200_MAX_STREAMS; ++s)
            if (s < n) x[s] = *reinterpret_cast<const float4 *>(xin + s * p.streams_in_stride + i);
        const float4 yv = *reinterpret_cast<const float4 *>(y + i);
        float4 u = make_float4(0, 0, 0, 0);
        for (int t = 0; t < n; ++t) {
            const float c = conn[n * n + t], take = conn[n * n + n + t];
            float4 a = make_float4(c * yv.x, c * yv.y, c * yv.z, c * yv.w);
#pragma unroll
            for (int s = 0; s < B200_MAX_STREAMS; ++s)
                if (s < n) {
                    const float w = conn[s * n + t];
                    a.x = fmaf(w, x[s].x, a.x); a.y = fmaf(w, x[s].y, a.y); a.z = fmaf(w, x[s].z, a.z); a.w = fmaf(w, x[s].w, a.w);
                }
            if (p.streams_out) *reinterpret_cast<float4 *>(p.streams_out + t * p.streams_out_stride + m * p.ld + i) = a;
            u.x = fmaf(take, a.x, u.x); u.y = fmaf(take, a.y, u.y); u.z = fmaf(take, a.z, u.z); u.w = fmaf(take, a.w, u.w);
        }
        if (p.u_out) *reinterpret_cast<float4 *>(p.u_out + m * p.ld + i) = u;
        *reinterpret_cast<float4 *>(row + i) = u;
        sum += (u.x + u.y) + (u.z + u.w);
    }
    if (!p.out) return;
    T *out = static_cast<T *>(p.out) + m * p.ld;
    layer_norm_row(row, sum, p.dim, p.ld, p.eps, p.gamma, p.beta, red, [&](int i, const float4 &v) { store4(out + i, v); });
}

template <typename T>
__global__ void __launch_bounds__(256) rows_start_kernel(const b200_rows_start_args p)
{
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const size_t m = blockIdx.x;
    uint32_t t = p.tokens[m];
    if (t >= (uint32_t)p.vocab) t = 0;                       // never outside the table
    const float *e = p.emb + (size_t)t * p.ld, *q = p.emb_pos + (size_t)min(p.pos0 + (int)m, p.pos_rows - 1) * p.ld;
    float sum = 0.0f;
    for (int i = 4 * threadIdx.x; i < p.ld; i += 1024) {
        const float4 a = *reinterpret_cast<const float4 *>(e + i), b = *reinterpret_cast<const float4 *>(q + i);
        const float4 v = make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w);
        *reinterpret_cast<float4 *>(row + i) = v;
        sum += (v.x + v.y) + (v.z + v.w);
    }
    const float take = *p.take;
    float *x = p.x + m * p.ld, next = 0.0f;
    layer_norm_row(row, sum, p.dim, p.ld, p.eps, p.emb_gamma, p.emb_beta, red, [&](int i, const float4 &v) {
        store4(x + i, v);
        const float4 u = make_float4(take * v.x, take * v.y, take * v.z, take * v.w);
        *reinterpret_cast<float4 *>(row + i) = u;            // this thread's own quad
        next += (u.x + u.y) + (u.z + u.w);
    });
    T *out = static_cast<T *>(p.out) + m * p.ld;
    layer_norm_row(row, next, p.dim, p.ld, p.eps, p.gamma, p.beta, red, [&](int i, const float4 &v) { store4(out + i, v); });
}

template <typename T>
__global__ void __launch_bounds__(256)
rows_layer_norm_kernel(const float *x, const int *index, int dim, int ld, float eps, const float *gamma, const float *beta, T *out)
{
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const size_t m = blockIdx.x, src = index ? (size_t)index[m] : m;
    float sum = 0.0f;
    for (int i = 4 * threadIdx.x; i < ld; i += 1024) {
        float4 v = *reinterpret_cast<const float4 *>(x + src * ld + i);
        float *e = &v.x;
#pragma unroll
        for (int k = 0; k < 4; ++k)
            if (i + k >= dim) e[k] = 0.0f;
        *reinterpret_cast<float4 *>(row + i) = v;
        sum += (v.x + v.y) + (v.z + v.w);
    }
    layer_norm_row(row, sum, dim, ld, eps, gamma, beta, red, [&](int i, const float4 &v) { store4(out + m * ld + i, v); });
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

static bool typed(int wtype) { return wtype == B200_WT_BF16 || wtype == B200_WT_F32; }

extern "C" int b200_rows_streams(const b200_rows_streams_args *a, void *stream)
{
    if (!a || !a->streams_in || !a->y || !a->connect || a->n_streams < 1 || a->n_streams > B200_MAX_STREAMS || a->rows <= 0 || a->dim <= 0 ||
        a->ld < a->dim || (a->ld & 3) || (a->y_ld & 3) || a->y_ld < a->ld || (a->streams_in_stride & 3) || (a->streams_out_stride & 3) ||
        (a->out && (!a->gamma || !a->beta || !typed(a->wtype))) || (!a->out && !a->streams_out && !a->u_out))
        return B200_E_BADARG;
    const size_t smem = (size_t)a->ld * 4;
    cudaStream_t st = (cudaStream_t)stream;
    int rc;
    if (a->wtype == B200_WT_F32) {
        if ((rc = row_smem(rows_streams_kernel<float>, smem)) != 0) return rc;
        rows_streams_kernel<float><<<a->rows, 256, smem, st>>>(*a);
    } else {
        if ((rc = row_smem(rows_streams_kernel<__nv_bfloat16>, smem)) != 0) return rc;
        rows_streams_kernel<__nv_bfloat16><<<a->rows, 256, smem, st>>>(*a);
    }
    return done();
}

extern "C" int b200_rows_start(const b200_rows_start_args *a, void *stream)
{
    if (!a || !a->emb || !a->emb_pos || !a->tokens || !a->emb_gamma || !a->emb_beta || !a->take || !a->gamma || !a->beta || !a->x || !a->out ||
        a->rows <= 0 || a->dim <= 0 || a->ld < a->dim || (a->ld & 3) || a->vocab <= 0 || a->pos_rows <= 0 || a->pos0 < 0 || !typed(a->wtype))
        return B200_E_BADARG;
    const size_t smem = (size_t)a->ld * 4;
    cudaStream_t st = (cudaStream_t)stream;
    int rc;
    if (a->wtype == B200_WT_F32) {
        if ((rc = row_smem(rows_start_kernel<float>, smem)) != 0) return rc;
        rows_start_kernel<float><<<a->rows, 256, smem, st>>>(*a);
    } else {
        if ((rc = row_smem(rows_start_kernel<__nv_bfloat16>, smem)) != 0) return rc;
        rows_start_kernel<__nv_bfloat16><<<a->rows, 256, smem, st>>>(*a);
    }
    return done();
}

extern "C" int b200_rows_layer_norm(const float *x, const int *index, int rows, int dim, int ld, float eps,
                                    const float *gamma, const float *beta, int wtype, void *out, void *stream)
{
    if (!x || !gamma || !beta || !out || rows <= 0 || dim <= 0 || ld < dim || (ld & 3) || !typed(wtype)) return B200_E_BADARG;
    const size_t smem = (size_t)ld * 4;
    cudaStream_t st = (cudaStream_t)stream;
    int rc;
    if (wtype == B200_WT_F32) {
        if ((rc = row_smem(rows_layer_norm_kernel<float>, smem)) != 0) return rc;
        rows_layer_norm_kernel<float><<<rows, 256, smem, st>>>(x, index, dim, ld, eps, gamma, beta, static_cast<float *>(out));
    } else {
        if ((rc = row_smem(rows_layer_norm_kernel<__nv_bfloat16>, smem)) != 0) return rc;
        rows_layer_norm_kernel<__nv_bfloat16><<<rows, 256, smem, st>>>(x, index, dim, ld, eps, gamma, beta, static_cast<__nv_bfloat16 *>(out));
    }
    return done();
}
