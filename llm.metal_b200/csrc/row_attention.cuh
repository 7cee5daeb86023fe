// Causal attention of many query rows over stored key and value rows (sm_100a), shared by the kinds of attention whose
// keys and values exist as rows: row_attend_bf16, tiled online softmax on the tensor cores (mma.sync m16n8k16, bfloat16
// operands, fp32 scores, weights and sums), and row_attend_f32, the same sum in fp32 on the CUDA cores.
#pragma once
#include "stream_core.cuh"
#include "../../include/llmb200_kernels.h"

#include <cuda_bf16.h>

extern unsigned long long g_b200_launches;

namespace {

__host__ __device__ __forceinline__ int up8(int n) { return (n + 7) & ~7; }

template <int WT> struct Elem;
template <> struct Elem<B200_WT_BF16> {
    using T = __nv_bfloat16;
    static constexpr int E = 8;
    static __device__ __forceinline__ float dot(const uint4 &w, const float *x) { return dot8_bf16(w, x); }
    static __device__ __forceinline__ void unpack(const uint4 &w, float *x)
    {
        const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = bf16_pair(u[i]); x[2 * i] = f.x; x[2 * i + 1] = f.y; }
    }
};
template <> struct Elem<B200_WT_F32> {
    using T = float;
    static constexpr int E = 4;
    static __device__ __forceinline__ float dot(const uint4 &w, const float *x) { return dot4_f32(w, x); }
    static __device__ __forceinline__ void unpack(const uint4 &w, float *x)
    {
        x[0] = __uint_as_float(w.x); x[1] = __uint_as_float(w.y); x[2] = __uint_as_float(w.z); x[3] = __uint_as_float(w.w);
    }
};

// Query row m (position pos0 + m) of head h sees key rows p with p <= pos0 + m and, with a window, pos0 + m - p < window.
// Head h reads key / value head h / group. score = scale * (q . k), or softcap * tanh of that over softcap.
struct RowAttn {
    int n_rows, pos0, heads, group, window;
    int dim, rot_dim, vdim;                  // a query row is [up8(dim) | up8(rot_dim)], padding zero
    float scale, softcap;                    // softcap 0: none
    const void *q;                           // [n_rows][heads] query rows
    const void *k; long long k_ld, k_head;   // first part of key row p of head g: k + g * k_head + (p - kv_row0) * k_ld
    const void *k2; long long k2_ld;         // second part (rot_dim > 0), one for all heads: k2 + p * k2_ld
    const void *v; long long v_ld, v_head;   // as k
    int kv_row0;
    const float *gate; long long gate_ld;    // results times sigmoid(gate), or NULL
    void *out; long long out_ld;             // [n_rows] rows of heads * vdim
};

__device__ __forceinline__ void cp16(uint32_t dst, const void *src, bool on)
{
    const int n = on ? 16 : 0;                               // 0: the 16 bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void ldsm4(uint32_t a, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4_t(uint32_t a, uint32_t (&r)[4])
{
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1)
{
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi)
{
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&h);
}

template <typename K>
int allow_smem(K kern, size_t smem)
{
    if (smem > 227 * 1024) return B200_E_TOOLARGE;
    return smem > 48 * 1024 ? (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : 0;
}

// fp32: one warp per (row, head), a lane per key, value columns over the lanes (256 per blockIdx.z).
__global__ void __launch_bounds__(128) row_attend_f32_kernel(const __grid_constant__ RowAttn p)
{
    extern __shared__ __align__(16) float qsh[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.y * 4 + warp, m = blockIdx.x, c0 = blockIdx.z * 256;
    if (h >= p.heads) return;                                // warps are independent of one another
    const int dim8 = up8(p.dim), QS = dim8 + up8(p.rot_dim);
    float *q = qsh + (size_t)warp * QS;
    const float *qg = static_cast<const float *>(p.q) + ((size_t)m * p.heads + h) * QS;
    for (int i = lane; i < QS; i += 32) q[i] = qg[i];
    __syncwarp();
    const int pos = p.pos0 + m;
    const int lo = p.window > 0 && pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
    const float *keys = static_cast<const float *>(p.k) + (h / p.group) * p.k_head, *values = static_cast<const float *>(p.v) + (h / p.group) * p.v_head;
    float mx = -INFINITY, l = 0.0f, acc[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) acc[c] = 0.0f;
    for (int k0 = lo; k0 <= pos; k0 += 32) {
        const int n = min(32, pos - k0 + 1), kp = k0 + lane;
        float s = -INFINITY;
        if (lane < n) {
            const float *kn = keys + (size_t)(kp - p.kv_row0) * p.k_ld, *kr = static_cast<const float *>(p.k2) + (size_t)kp * p.k2_ld;
            float a = 0.0f, b = 0.0f;
            for (int d = 0; d < p.dim; ++d) a = fmaf(q[d], kn[d], a);
            for (int d = 0; d < p.rot_dim; ++d) b = fmaf(q[dim8 + d], kr[d], b);
            s = p.scale * (a + b);
            if (p.softcap > 0.0f) s = p.softcap * tanhf(s / p.softcap);
        }
        const float mt = fmaxf(mx, warp_max(s));
        const float w = lane < n ? expf(s - mt) : 0.0f;
        const float corr = mx == -INFINITY ? 0.0f : expf(mx - mt);
        l = l * corr + warp_sum(w);
        mx = mt;
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[c] *= corr;
        for (int j = 0; j < n; ++j) {
            const float wj = __shfl_sync(0xffffffffu, w, j);
            const float *v = values + (size_t)(k0 + j - p.kv_row0) * p.v_ld;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                const int col = c0 + c * 32 + lane;
                if (col < p.vdim) acc[c] = fmaf(wj, v[col], acc[c]);
            }
        }
    }
    const float inv = 1.0f / l;
    float *o = static_cast<float *>(p.out) + (size_t)m * p.out_ld + (size_t)h * p.vdim;
    const float *gate = p.gate ? p.gate + (size_t)m * p.gate_ld + (size_t)h * p.vdim : nullptr;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
        const int col = c0 + c * 32 + lane;
        if (col < p.vdim) o[col] = acc[c] * inv * (gate ? sigmoid_f32(gate[col]) : 1.0f);
    }
}

// bfloat16 on the tensor cores. A block: NW warps of 16 query rows of one head; keys 32 at a time, the next tile's
// copies in flight under the current one. DV value columns per blockIdx.z.
constexpr int BKEY = 32;

__device__ __forceinline__ float ex2(float x)                // 2^x, 2 ulp, 0 for -inf
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// cap * tanh(s / cap) through one exponential: exact at both ends, absolute error a few cap * 2^-24
__device__ __forceinline__ float soft_cap(float s, float two_log2e_over_cap, float cap)
{
    return cap - __fdividef(2.0f * cap, ex2(s * two_log2e_over_cap) + 1.0f);
}
// Later rows see more keys. Blocks are numbered from the heaviest tile of rows to the lightest; where two of them share
// an SM and all are resident at once, the second half counts from the light end, so that every SM gets about the same.
struct Place { int tile, head; };
__device__ __forceinline__ Place place_of(int id, int n, int heads, int wave)
{
    const int r = id < wave || n > 2 * wave ? id : n - 1 - (id - wave);
    return {n / heads - 1 - r / heads, r % heads};
}

template <int DV, int NW, bool CAP>
__global__ void __launch_bounds__(NW * 32, 16 / NW) row_attend_bf16_kernel(const __grid_constant__ RowAttn p, int dqs, int stages, int wave)
{
    // dqs: elements of a query / key row in shared memory; its first dqs - 8 are multiples of 16 and hold
    // [unrotated | rotated | zeros]. Rows are 16 bytes off a multiple of 32: ldmatrix is conflict-free.
    constexpr int VS = DV + 8, BQ = NW * 16, NT = NW * 32;
    extern __shared__ __align__(16) unsigned char smem[];
    const int dim8 = up8(p.dim), QS = dim8 + up8(p.rot_dim), vd8 = up8(p.vdim);
    const int dqk = dqs - 8;
    __nv_bfloat16 *qsm = reinterpret_cast<__nv_bfloat16 *>(smem);
    __nv_bfloat16 *ksm = qsm + (size_t)BQ * dqs;             // [stages][BKEY][dqs]
    __nv_bfloat16 *vsm = ksm + (size_t)stages * BKEY * dqs;  // [stages][BKEY][VS]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const Place place = place_of(blockIdx.x, gridDim.x, p.heads, wave);
    const int h = place.head, m0 = place.tile * BQ, c0 = blockIdx.y * DV;
    const int rows = min(BQ, p.n_rows - m0);
    const __nv_bfloat16 *keys = static_cast<const __nv_bfloat16 *>(p.k) + (h / p.group) * p.k_head;
    const __nv_bfloat16 *values = static_cast<const __nv_bfloat16 *>(p.v) + (h / p.group) * p.v_head;
    const __nv_bfloat16 *qg = static_cast<const __nv_bfloat16 *>(p.q) + ((size_t)m0 * p.heads + h) * QS;

    const int first = p.pos0 + m0, last = first + rows - 1;  // absolute positions of this block's queries
    const int lo = p.window > 0 && first - p.window + 1 > 0 ? first - p.window + 1 : 0;
    const int tiles = (last - lo) / BKEY + 1;
    const int sq = dqk / 8;
    constexpr int SV = DV / 8;
    // 16-byte chunks of a [rows][sq] tile go round the threads: (row, chunk) of this thread and its step, no divisions
    const int r_first = tid / sq, c_first = tid % sq, r_step = NT / sq, c_step = NT % sq;

    for (int r = r_first, c = c_first; r < BQ;) {
        const bool on = r < rows && c * 8 < QS;
        cp16(smem_u32(qsm + r * dqs + c * 8), on ? qg + (size_t)r * p.heads * QS + c * 8 : qg, on);
        r += r_step; c += c_step;
        if (c >= sq) { c -= sq; ++r; }
    }
    auto stage = [&](int tile, int slot) {
        const uint32_t kd = smem_u32(ksm + slot * BKEY * dqs), vd = smem_u32(vsm + slot * BKEY * VS);
        const int k0 = lo + tile * BKEY, n = last - k0;      // rows past n hold zeros
        const __nv_bfloat16 *kt = keys + (long long)(k0 - p.kv_row0) * p.k_ld, *vt = values + (long long)(k0 - p.kv_row0) * p.v_ld;
        const __nv_bfloat16 *k2t = static_cast<const __nv_bfloat16 *>(p.k2) + (long long)k0 * p.k2_ld - dim8;
        for (int r = r_first, c = c_first; r < BKEY;) {
            const bool on = r <= n && c * 8 < QS;
            const __nv_bfloat16 *src = c * 8 < dim8 ? kt + (long long)r * p.k_ld : k2t + (long long)r * p.k2_ld;
            cp16(kd + (r * dqs + c * 8) * 2, on ? src + c * 8 : keys, on);
            r += r_step; c += c_step;
            if (c >= sq) { c -= sq; ++r; }
        }
#pragma unroll
        for (int i = 0; i < (BKEY * SV + NT - 1) / NT; ++i) {
            const int e = tid + i * NT, r = e / SV, c = e % SV;
            if (BKEY * SV % NT == 0 || r < BKEY) {
                const bool on = r <= n && c0 + c * 8 < vd8;
                cp16(vd + (r * VS + c * 8) * 2, on ? vt + (long long)r * p.v_ld + c0 + c * 8 : keys, on);
            }
        }
        cp_commit();
    };
    stage(0, 0);

    float o[DV / 8][4];
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) o[i][k] = 0.0f;
    float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};      // maxima of the unscaled (or capped) scores
    // this thread's rows: r0 and r0 + 8 of the warp's 16
    const int r0 = warp * 16 + (lane >> 2);
    const uint32_t qaddr = smem_u32(qsm + (warp * 16 + (lane & 15)) * dqs + (lane >> 4) * 8);
    const float sc = (CAP ? 1.0f : p.scale) * 1.4426950408889634f;          // weights as powers of two
    const float cap_in = CAP ? 2.0f * 1.4426950408889634f * p.scale / p.softcap : 0.0f;

    for (int tile = 0; tile < tiles; ++tile) {
        const int slot = stages == 2 ? tile & 1 : 0;
        if (stages == 2 && tile + 1 < tiles) {
            stage(tile + 1, slot ^ 1);
            cp_wait<1>();
        } else {
            cp_wait<0>();
        }
        __syncthreads();
        const int k0 = lo + tile * BKEY;
        // the warp's queries see nothing of this tile: all of it is ahead of them, or has left their windows
        const int w_first = first + warp * 16, w_last = w_first + 15;
        const bool idle = k0 > w_last || (p.window > 0 && w_first - (k0 + BKEY - 1) >= p.window);
        if (!idle) {
            float s[BKEY / 8][4];
#pragma unroll
            for (int i = 0; i < BKEY / 8; ++i)
#pragma unroll
                for (int k = 0; k < 4; ++k) s[i][k] = 0.0f;
            // key rows as the B operand: matrices (keys 0-7, k 0-7), (keys 0-7, k 8-15), (keys 8-15, k 0-7), (keys 8-15, k 8-15)
            const uint32_t kaddr = smem_u32(ksm + slot * BKEY * dqs + ((lane & 7) + ((lane >> 4) << 3)) * dqs + ((lane >> 3) & 1) * 8);
#pragma unroll 4
            for (int kk = 0; kk < dqk; kk += 16) {
                uint32_t a[4];
                ldsm4(qaddr + kk * 2, a);
#pragma unroll
                for (int n = 0; n < BKEY / 16; ++n) {
                    uint32_t b[4];
                    ldsm4(kaddr + (uint32_t)(n * 16 * dqs + kk) * 2, b);
                    mma_bf16(s[2 * n], a, b[0], b[1]);
                    mma_bf16(s[2 * n + 1], a, b[2], b[3]);
                }
            }
            if constexpr (CAP) {
#pragma unroll
                for (int n = 0; n < BKEY / 8; ++n)
#pragma unroll
                    for (int k = 0; k < 4; ++k) s[n][k] = soft_cap(s[n][k], cap_in, p.softcap);
            }
            // only tiles at an edge of the warp's visible range need the mask
            if (k0 + BKEY - 1 > w_first || (p.window > 0 && w_last - k0 >= p.window)) {
                const int span = p.window > 0 ? p.window : 0x7fffffff;
                const int d0 = first + r0 - k0 - (lane & 3) * 2;
#pragma unroll
                for (int n = 0; n < BKEY / 8; ++n)
#pragma unroll
                    for (int k = 0; k < 4; ++k) {
                        const int d = d0 + (k >> 1) * 8 - n * 8 - (k & 1);
                        if (d < 0 || d >= span) s[n][k] = -INFINITY;
                    }
            }
            float mt[2] = {mx[0], mx[1]};
#pragma unroll
            for (int n = 0; n < BKEY / 8; ++n) {
                mt[0] = fmaxf(mt[0], fmaxf(s[n][0], s[n][1]));
                mt[1] = fmaxf(mt[1], fmaxf(s[n][2], s[n][3]));
            }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 1));
                mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 2));
            }
            // a row with nothing visible so far keeps its maximum at -inf: its weights and its correction are zero
            // (differences first: the score at the maximum then weighs exactly one, whatever its size)
            const float base[2] = {mt[0] == -INFINITY ? 0.0f : mt[0], mt[1] == -INFINITY ? 0.0f : mt[1]};
            const float corr[2] = {ex2((mx[0] - base[0]) * sc), ex2((mx[1] - base[1]) * sc)};
            const bool moved = mt[0] != mx[0] || mt[1] != mx[1];
            mx[0] = mt[0]; mx[1] = mt[1];
            float ls[2] = {0.0f, 0.0f};
#pragma unroll
            for (int n = 0; n < BKEY / 8; ++n)
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    s[n][k] = ex2((s[n][k] - base[k >> 1]) * sc);
                    ls[k >> 1] += s[n][k];
                }
            l[0] = fmaf(l[0], corr[0], ls[0]);
            l[1] = fmaf(l[1], corr[1], ls[1]);
            if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
                for (int i = 0; i < DV / 8; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
            }
            // value rows as the B operand, transposed on load: (k 0-7, cols 0-7), (k 8-15, cols 0-7), (k 0-7, cols 8-15), ...
            const uint32_t vaddr = smem_u32(vsm + slot * BKEY * VS + (lane & 15) * VS + (lane >> 4) * 8);
#pragma unroll
            for (int kk = 0; kk < BKEY / 16; ++kk) {
                const uint32_t a[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                       pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
                for (int n = 0; n < DV / 16; ++n) {
                    uint32_t b[4];
                    ldsm4_t(vaddr + (uint32_t)(kk * 16 * VS + n * 16) * 2, b);
                    mma_bf16(o[2 * n], a, b[0], b[1]);
                    mma_bf16(o[2 * n + 1], a, b[2], b[3]);
                }
            }
        }
        __syncthreads();                                     // the slot is overwritten by the next round's copies
        if (stages == 1 && tile + 1 < tiles) stage(tile + 1, 0);
    }

#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        if (r0 + 8 * r >= rows) continue;
        const float inv = 1.0f / l[r];
        const size_t m = (size_t)(m0 + r0 + 8 * r);
        __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.out) + m * p.out_ld + (size_t)h * p.vdim;
        const float *gate = p.gate ? p.gate + m * p.gate_ld + (size_t)h * p.vdim : nullptr;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i)
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int col = c0 + i * 8 + (lane & 3) * 2 + k;
                if (col < p.vdim) out[col] = __float2bfloat16_rn(o[i][2 * r + k] * inv * (gate ? sigmoid_f32(gate[col]) : 1.0f));
            }
    }
}

template <int DV, int NW, bool CAP>
int row_attend_bf16(const RowAttn &a, cudaStream_t st)
{
    const int dqk = (up8(a.dim) + up8(a.rot_dim) + 15) / 16 * 16, dqs = dqk + 8;
    int stages = 2;
    auto bytes = [&](int s) { return ((size_t)(NW * 16 + s * BKEY) * dqs + (size_t)s * BKEY * (DV + 8)) * 2; };
    if (bytes(2) > 227 * 1024) stages = 1;
    int rc = allow_smem(row_attend_bf16_kernel<DV, NW, CAP>, bytes(stages));
    if (rc) return rc;
    const dim3 grid((a.n_rows + NW * 16 - 1) / (NW * 16) * a.heads, (a.vdim + DV - 1) / DV);
    row_attend_bf16_kernel<DV, NW, CAP><<<grid, NW * 32, bytes(stages), st>>>(a, dqs, stages, 148);
    ++g_b200_launches;
    return (int)cudaGetLastError();
}

// 128 query rows a block where that still fills the machine (a tile of keys serves twice the rows), 64 otherwise
template <int DV, bool CAP>
int row_attend_bf16(const RowAttn &a, cudaStream_t st)
{
    return (long long)((a.n_rows + 127) / 128) * a.heads >= 148 ? row_attend_bf16<DV, 8, CAP>(a, st) : row_attend_bf16<DV, 4, CAP>(a, st);
}

template <bool CAP>
int row_attend_bf16(const RowAttn &a, cudaStream_t st)
{
    if (a.vdim <= 32) return row_attend_bf16<32, CAP>(a, st);
    if (a.vdim <= 64) return row_attend_bf16<64, CAP>(a, st);
    return row_attend_bf16<128, CAP>(a, st);
}

int row_attend_f32(const RowAttn &a, cudaStream_t st)
{
    const size_t smem = (size_t)4 * (up8(a.dim) + up8(a.rot_dim)) * 4;
    const int rc = allow_smem(row_attend_f32_kernel, smem);
    if (rc) return rc;
    row_attend_f32_kernel<<<dim3(a.n_rows, (a.heads + 3) / 4, (a.vdim + 255) / 256), 128, smem, st>>>(a);
    ++g_b200_launches;
    return (int)cudaGetLastError();
}

}  // namespace
