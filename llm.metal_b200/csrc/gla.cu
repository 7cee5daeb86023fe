// Gated linear attention (sm_100a): per head a state S [dim][vdim] that decays by a factor per key channel and takes in
// one outer product per token, everything from the projections on in fp32 (the products over chunks of a prompt on the
// tensor cores, every fp32 operand as a sum of three bfloat16 numbers, 24 significant bits, with fp32 sums).
//
// Decode, one launch: a cluster of blocks per head, each block a slice of the columns. The state slice and the weights
// of the decay are fetched before the kernel waits for its predecessor; the norm over a head's result is a sum across
// the cluster through distributed shared memory.
//
// Prompt portions: chunks of 64 tokens in parallel. With c_t the running sum of the log decays inside a chunk,
//   o_t = (q_t exp(c_t)) S_in + sum over s <= t of (sum over channels q_t k_s exp(c_t - c_s)) v_s
//   S_out = exp(c_end) S_in + sum over s of (k_s exp(c_end - c_s)) v_s^T
// gla_prep forms the decayed queries and keys and the score matrix, and splits them and the values into three bfloat16
// planes for the products that follow; gla_states walks the chunks with a tile of the state
// in registers and leaves the state before each (split as well), gla_out forms the outputs. Every exponent that is taken is <= 0: inside
// eight tokens the differences c_t - c_s are exponentiated pair by pair, across eights and sixteens as a product through
// the value of c between the two.
#include "stream_core.cuh"
#include "../../include/llmb200_kernels.h"

#include <cooperative_groups.h>
#include <cuda_bf16.h>

extern unsigned long long g_b200_launches;

namespace cg = cooperative_groups;

namespace {

constexpr int C = B200_GLA_CHUNK, SUB = 16;
constexpr int THREADS = 256;
constexpr int MAX_CLUSTER = 8;

__host__ __device__ __forceinline__ int up4(int n) { return (n + 3) & ~3; }
__host__ __device__ __forceinline__ int up8(int n) { return (n + 7) & ~7; }
__host__ __device__ __forceinline__ int up16(int n) { return (n + 15) & ~15; }

// log(logistic(z)), no overflow on either side
__device__ __forceinline__ float log_logistic(float z) { return fminf(z, 0.0f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_f32(float z) { return z * sigmoid_f32(z); }

// A decay factor exp(x), x <= 0, as the pair (m, keep) for S <- keep S + (m S + u). Near one the factor's own rounding,
// the same for every token of a slow channel, would add up over hundreds of tokens, so there m = exp(x) - 1 and keep = 1;
// elsewhere m = exp(x) and keep = 0.
struct Decay { float m, keep; };
__device__ __forceinline__ Decay decay_of(float x)
{
    const float m = expm1f(x);
    return m > -0.5f ? Decay{m, 1.0f} : Decay{expf(x), 0.0f};
}
__device__ __forceinline__ float decayed(float s, const Decay &a, float u) { return fmaf(a.keep, s, fmaf(a.m, s, u)); }

__device__ __forceinline__ float dot4(const float4 &a, const float4 &b, float acc)
{
    return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, acc))));
}

__device__ __forceinline__ void cp16(void *dst, const void *src)
{
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// ------------------------------------------------------------------------------------------------ decode

// vg: quads of columns a block covers (a power of two <= 32); a thread owns one quad of every THREADS / vg -th row.
__global__ void __launch_bounds__(THREADS) gla_decode_kernel(const __grid_constant__ b200_gla_args p, int vg, int cluster_size)
{
    constexpr int HELD = 8;                                  // rows a thread holds before the wait
    extern __shared__ __align__(16) float sh[];
    __shared__ float red[33], part_ss[MAX_CLUSTER];
    pdl_launch_dependents();
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int h = blockIdx.x / cluster_size, rank = blockIdx.x % cluster_size;
    const int dim = p.dim, v8 = up8(p.vdim), R4 = up4(p.rank), w16 = (R4 / 4) | 1;      // odd: rows 16 bytes apart mod 32
    const int VW = 4 * vg, c0 = rank * VW, RG = THREADS / vg, rg = tid / vg, col = c0 + 4 * (tid % vg);
    Decay *sa = reinterpret_cast<Decay *>(sh);
    float *sk = sh + 2 * up4(dim), *sq = sk + up4(dim), *so = sq + up4(dim), *w2 = so + (THREADS / 32) * VW;
    const int pos = *p.d_pos;
    const size_t slot = (size_t)p.heads * dim * v8;
    const float *s_in = p.d_state + (size_t)(max(pos, 0) % p.n_slots) * slot + (size_t)h * dim * v8;
    float *s_out = p.d_state + (size_t)((max(pos, 0) + 1) % p.n_slots) * slot + (size_t)h * dim * v8;
    const bool fresh = pos <= 0, mine = col < v8;
    const float4 zero = make_float4(0, 0, 0, 0);

    float4 st[HELD];
#pragma unroll
    for (int i = 0; i < HELD; ++i) {
        const int d = rg + i * RG;
        st[i] = mine && !fresh && d < dim ? *reinterpret_cast<const float4 *>(s_in + (size_t)d * v8 + col) : zero;
    }
    for (int e = tid; e < dim * (R4 / 4); e += THREADS) {
        const int d = e / (R4 / 4), c = e % (R4 / 4);
        cp16(w2 + ((size_t)d * w16 + c) * 4, p.d_a2 + ((size_t)h * dim + d) * R4 + c * 4);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");     // every block of the cluster has started
    const float bias0 = tid < dim ? p.d_a2_bias[h * dim + tid] : 0.0f;
    const float gamma = tid < VW && c0 + tid < p.vdim ? p.d_norm_gamma[c0 + tid] : 0.0f;
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    pdl_wait();

    const float gate = tid < VW && c0 + tid < p.vdim ? p.d_gate[h * p.vdim + c0 + tid] : 0.0f;
    float4 v = zero;
    if (mine) {
        const float *vp = p.d_v + h * p.vdim + col;
        v.x = col < p.vdim ? vp[0] : 0.0f; v.y = col + 1 < p.vdim ? vp[1] : 0.0f;
        v.z = col + 2 < p.vdim ? vp[2] : 0.0f; v.w = col + 3 < p.vdim ? vp[3] : 0.0f;
    }
    for (int d = tid; d < dim; d += THREADS) {
        const float k = p.d_k[h * dim + d], q = p.d_q[h * dim + d];
        float z = d == tid ? bias0 : p.d_a2_bias[h * dim + d];
        for (int c = 0; c < R4 / 4; ++c)
            z = dot4(*reinterpret_cast<const float4 *>(w2 + ((size_t)d * w16 + c) * 4), *reinterpret_cast<const float4 *>(p.d_f + 4 * c), z);
        sa[d] = decay_of(log_logistic(z) / p.tau);
        sk[d] = k;
        sq[d] = q * p.q_scale;
    }
    __syncthreads();
    float4 o = zero;
    auto step = [&](float4 s, int d) {
        const Decay a = sa[d];
        const float k = sk[d], q = sq[d];
        s.x = decayed(s.x, a, k * v.x); s.y = decayed(s.y, a, k * v.y); s.z = decayed(s.z, a, k * v.z); s.w = decayed(s.w, a, k * v.w);
        *reinterpret_cast<float4 *>(s_out + (size_t)d * v8 + col) = s;
        o.x = fmaf(q, s.x, o.x); o.y = fmaf(q, s.y, o.y); o.z = fmaf(q, s.z, o.z); o.w = fmaf(q, s.w, o.w);
    };
    if (mine) {
#pragma unroll
        for (int i = 0; i < HELD; ++i)
            if (rg + i * RG < dim) step(st[i], rg + i * RG);
        for (int d0 = rg + HELD * RG; d0 < dim; d0 += HELD * RG) {
#pragma unroll
            for (int i = 0; i < HELD; ++i) {
                const int d = d0 + i * RG;
                st[i] = !fresh && d < dim ? *reinterpret_cast<const float4 *>(s_in + (size_t)d * v8 + col) : zero;
            }
#pragma unroll
            for (int i = 0; i < HELD; ++i)
                if (d0 + i * RG < dim) step(st[i], d0 + i * RG);
        }
    }
    for (int x = vg; x < 32; x <<= 1) {
        o.x += __shfl_xor_sync(0xffffffffu, o.x, x); o.y += __shfl_xor_sync(0xffffffffu, o.y, x);
        o.z += __shfl_xor_sync(0xffffffffu, o.z, x); o.w += __shfl_xor_sync(0xffffffffu, o.w, x);
    }
    if (lane < vg) *reinterpret_cast<float4 *>(so + warp * VW + 4 * lane) = o;
    __syncthreads();
    float y = 0.0f;
    if (tid < VW) {
#pragma unroll
        for (int w = 0; w < THREADS / 32; ++w) y += so[w * VW + tid];
        if (c0 + tid >= p.vdim) y = 0.0f;
    }
    const float ss = block_sum(y * y, red);
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (tid < cluster_size) *cluster.map_shared_rank(&part_ss[rank], tid) = ss;
    cluster.sync();
    float total = 0.0f;
    for (int r = 0; r < cluster_size; ++r) total += part_ss[r];
    const float inv = 1.0f / sqrtf(total / (float)p.vdim + p.eps);
    if (tid < VW && c0 + tid < p.vdim) p.d_out[h * p.vdim + c0 + tid] = gamma * (y * inv) * silu_f32(gate);
}

// ------------------------------------------------------------------------------------------------ rows

constexpr int DT = 32, RS = DT + 4;                          // channels of a pass; row of a tile: 16 bytes off a multiple of 32
constexpr int EIGHT_PAIRS = 36, N_PAIRS = C / 8 * EIGHT_PAIRS;       // s <= t inside eight tokens; of a chunk

// x = hi + mid + lo, each the nearest bfloat16 of what is left; stored `plane` elements apart.
__device__ __forceinline__ void put_split(__nv_bfloat16 *out, size_t plane, float x)
{
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const __nv_bfloat16 h = __float2bfloat16_rn(x);
        out[k * plane] = h;
        x -= __bfloat162float(h);
    }
}
// Two tokens' values of this lane's channel: neighbouring lanes swap one each, so that the even lane stores both channels
// of the first token and the odd lane both of the second. out: the first token's even channel; ld: elements to the second.
__device__ __forceinline__ void put_split2(__nv_bfloat16 *out, size_t plane, float x, float y);
__device__ __forceinline__ void put_split_pair(__nv_bfloat16 *out, int ld, size_t plane, float first, float second, bool on)
{
    const bool odd = threadIdx.x & 1;
    const float other = __shfl_xor_sync(0xffffffffu, odd ? first : second, 1);
    if (on) put_split2(out + (odd ? ld : 0), plane, odd ? other : first, odd ? second : other);
}
__device__ __forceinline__ void put_split2(__nv_bfloat16 *out, size_t plane, float x, float y)       // two neighbours, 4-byte aligned
{
#pragma unroll
    for (int k = 0; k < 3; ++k) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
        const uint32_t w = *reinterpret_cast<const uint32_t *>(&h);
        *reinterpret_cast<uint32_t *>(out + k * plane) = w;
        const float2 f = bf16_pair(w);
        x -= f.x;
        y -= f.y;
    }
}

// The pair (t, s) number e of a chunk's eights.
__device__ __forceinline__ void pair_of(int e, int &t, int &s)
{
    const int base = e / EIGHT_PAIRS * 8;
    int k = e % EIGHT_PAIRS, row = 0;
    while (k > row) { k -= row + 1; ++row; }
    t = base + row;
    s = base + k;
}
__device__ __forceinline__ float score4(const float4 &q, const float4 &k, const float4 &ct, const float4 &cs, float acc)
{
    const float4 w = make_float4(exp2f(ct.x - cs.x), exp2f(ct.y - cs.y), exp2f(ct.z - cs.z), exp2f(ct.w - cs.w));
    return dot4(make_float4(q.x * k.x, q.y * k.y, q.z * k.z, q.w * k.w), w, acc);
}
__device__ __forceinline__ float4 row4(const float *tile, int row, int col) { return *reinterpret_cast<const float4 *>(tile + row * RS + col); }

// One block per chunk and head. Shared: f [C][R4], then tiles of rows RS apart: c (running log2 of the decay), q, k [C];
// q from the start of its sixteen [C]; k up to the starts of the second, third and fourth sixteen [16 + 32 + 48]; q of the
// second eights and k of the first eights through the boundary between them [32] each.
__global__ void __launch_bounds__(THREADS) gla_prep_kernel(const __grid_constant__ b200_gla_args p)
{
    extern __shared__ __align__(16) float sh[];
    __shared__ float tot[8][DT];
    const int R4 = up4(p.rank), d8 = up8(p.dim), d16 = up16(p.dim), v8 = up8(p.vdim), tid = threadIdx.x;
    float *fs = sh, *cs = fs + C * R4, *qs = cs + C * RS, *ks = qs + C * RS, *qh = ks + C * RS, *kh = qh + C * RS;
    float *q8 = kh + 96 * RS, *k8 = q8 + C / 2 * RS, *ws = k8 + C / 2 * RS;
    const int chunk = blockIdx.x, h = blockIdx.y, m0 = chunk * C, n = min(C, p.n_rows - m0);
    const size_t ch = (size_t)chunk * p.heads + h;
    const int w16 = (R4 / 4) | 1;
    for (int e = tid; e < C * R4; e += THREADS) {
        const int t = e / R4, r = e % R4;
        fs[e] = t < n && r < p.rank ? p.d_f[(size_t)(m0 + t) * p.proj_ld + r] : 0.0f;
    }
    __nv_bfloat16 *const qd = static_cast<__nv_bfloat16 *>(p.d_qd) + ch * 3 * C * d16, *const kd = static_cast<__nv_bfloat16 *>(p.d_kd) + ch * 3 * C * d16;
    __nv_bfloat16 *const values = static_cast<__nv_bfloat16 *>(p.d_values) + ch * 3 * C * v8;
    // (loads that no store of this kernel can change are marked as such, or they would wait for the stores before them)
    const int step_t = THREADS / (v8 / 2 < THREADS ? v8 / 2 : THREADS);
    for (int j = tid % (THREADS / step_t) * 2; j < v8 && tid < step_t * (THREADS / step_t); j += THREADS * 2)
#pragma unroll 8
        for (int t = tid / (THREADS / step_t); t < C; t += step_t) {
            const float *v = p.d_v + (size_t)(m0 + t) * p.proj_ld + (size_t)h * p.vdim + j;
            put_split2(values + (size_t)t * v8 + j, (size_t)C * v8, t < n && j < p.vdim ? __ldg(v) : 0.0f, t < n && j + 1 < p.vdim ? __ldg(v + 1) : 0.0f);
        }
    // this thread's scores: one of every pair of sixteens i > j, one across the eights of a sixteen, one or two pairs of an eight
    const int ti = tid / SUB, si = tid % SUB;
    const int et = tid / 8 % 8, es = tid % 8, eb = tid / 64;
    int pt[2], ps[2];
    pair_of(tid, pt[0], ps[0]);
    pair_of(min(THREADS + tid, N_PAIRS - 1), pt[1], ps[1]);
    const bool two = THREADS + tid < N_PAIRS;
    float far[6], mid = 0.0f, near[2] = {0.0f, 0.0f};
#pragma unroll
    for (int x = 0; x < 6; ++x) far[x] = 0.0f;

    for (int d0 = 0; d0 < p.dim; d0 += DT) {
        __syncthreads();
        for (int e = tid; e < DT * (R4 / 4); e += THREADS) {
            const int d = e / (R4 / 4), c = e % (R4 / 4);
            *reinterpret_cast<float4 *>(ws + ((size_t)d * w16 + c) * 4) =
                d0 + d < p.dim ? *reinterpret_cast<const float4 *>(p.d_a2 + ((size_t)h * p.dim + d0 + d) * R4 + c * 4) : make_float4(0, 0, 0, 0);
        }
        const int d = tid % DT, tg = tid / DT;               // a channel, eight tokens
        const bool on = d0 + d < p.dim;
        float q[8], k[8], c[8];
        {
            const size_t at = (size_t)h * p.dim + d0 + d;
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int t = tg * 8 + i;
                q[i] = on && t < n ? __ldg(p.d_q + (size_t)(m0 + t) * p.proj_ld + at) * p.q_scale : 0.0f;
                k[i] = on && t < n ? __ldg(p.d_k + (size_t)(m0 + t) * p.proj_ld + at) : 0.0f;
            }
        }
        const float bias = on ? p.d_a2_bias[(size_t)h * p.dim + d0 + d] : 0.0f;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) c[i] = bias;
        for (int r = 0; r < R4 / 4; ++r) {
            const float4 w = *reinterpret_cast<const float4 *>(ws + ((size_t)d * w16 + r) * 4);
#pragma unroll
            for (int i = 0; i < 8; ++i) c[i] = dot4(w, *reinterpret_cast<const float4 *>(fs + (tg * 8 + i) * R4 + 4 * r), c[i]);
        }
        float run = 0.0f;
        const float unit = 1.4426950408889634f / p.tau;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (on && tg * 8 + i < n) run += log_logistic(c[i]) * unit;
            c[i] = run;
        }
        tot[tg][d] = run;
        __syncthreads();
        float before = 0.0f, end = 0.0f;
#pragma unroll
        for (int g = 0; g < 8; ++g) { if (g < tg) before += tot[g][d]; end += tot[g][d]; }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = tg * 8 + i;
            c[i] += before;
            cs[t * RS + d] = c[i]; qs[t * RS + d] = q[i]; ks[t * RS + d] = k[i];
        }
#pragma unroll
        for (int i = 0; i < 8; i += 2) {
            const size_t at = (size_t)(tg * 8 + i) * d16 + d0 + (d & ~1);
            put_split_pair(qd + at, d16, (size_t)C * d16, q[i] * exp2f(c[i]), q[i + 1] * exp2f(c[i + 1]), d0 + d < d16);
            put_split_pair(kd + at, d16, (size_t)C * d16, k[i] * exp2f(end - c[i]), k[i + 1] * exp2f(end - c[i + 1]), d0 + d < d16);
        }
        if (d0 + d < d8 && tg == 0) p.d_decay[ch * d8 + d0 + d] = end;
        __syncthreads();
        {   // through the boundaries: c just before each sixteen, c at the end of each first eight (this thread's tokens are one eight)
            const int u = tg / 2;
            const float start = u > 0 ? cs[(u * SUB - 1) * RS + d] : 0.0f, half = cs[(u * SUB + 7) * RS + d];
            float next[3];
#pragma unroll
            for (int v = 1; v < 4; ++v) next[v - 1] = cs[(v * SUB - 1) * RS + d];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                const int t = tg * 8 + i;
                if (u > 0) qh[t * RS + d] = q[i] * exp2f(c[i] - start);
                if (tg & 1) q8[(u * 8 + i) * RS + d] = q[i] * exp2f(c[i] - half);
                else k8[(u * 8 + i) * RS + d] = k[i] * exp2f(half - c[i]);
#pragma unroll
                for (int v = 1; v < 4; ++v)
                    if (u < v) kh[(v * (v - 1) * SUB / 2 + t) * RS + d] = k[i] * exp2f(next[v - 1] - c[i]);
            }
        }
        __syncthreads();
#pragma unroll 2
        for (int x = 0; x < DT; x += 4) {
#pragma unroll
            for (int i = 1, at = 0; i < 4; ++i) {
                const float4 a = row4(qh, i * SUB + ti, x);
#pragma unroll
                for (int j = 0; j < i; ++j, ++at) far[at] = dot4(a, row4(kh, i * (i - 1) * SUB / 2 + j * SUB + si, x), far[at]);
            }
            mid = dot4(row4(q8, eb * 8 + et, x), row4(k8, eb * 8 + es, x), mid);
            near[0] = score4(row4(qs, pt[0], x), row4(ks, ps[0], x), row4(cs, pt[0], x), row4(cs, ps[0], x), near[0]);
            if (two) near[1] = score4(row4(qs, pt[1], x), row4(ks, ps[1], x), row4(cs, pt[1], x), row4(cs, ps[1], x), near[1]);
        }
    }
    // zeros where s > t
    __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.d_scores) + ch * 3 * C * C;
    auto put = [&](int t, int s, float x) { put_split(out + t * C + s, C * C, x); };
#pragma unroll
    for (int i = 0, at = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (i > j) put(i * SUB + ti, j * SUB + si, far[at++]);
            else if (i < j) put(i * SUB + ti, j * SUB + si, 0.0f);
        }
    put(eb * SUB + 8 + et, eb * SUB + es, mid);
    put(eb * SUB + et, eb * SUB + 8 + es, 0.0f);
    put(pt[0], ps[0], near[0]);
    if (pt[0] != ps[0]) put(ps[0], pt[0], 0.0f);
    if (two) {
        put(pt[1], ps[1], near[1]);
        if (pt[1] != ps[1]) put(ps[1], pt[1], 0.0f);
    }
}

__device__ __forceinline__ void cp16_if(uint32_t dst, const void *src, bool on)
{
    const int n = on ? 16 : 0;                               // 0: zero-filled
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

// Three planes of ROWS x COLS elements to shared rows LD elements apart (planes ROWS * LD apart); rows from n_rows on and
// columns from n_cols on are zeros. src: row 0, column 0 of the first plane; its rows are ld, its planes `plane` apart.
template <int ROWS, int COLS, int LD, int NT>
__device__ __forceinline__ void fetch_planes(uint32_t dst, const __nv_bfloat16 *src, size_t plane, int ld, int n_rows, int n_cols)
{
    constexpr int PER = COLS / 8, STEP = NT / PER;           // pieces of a row; rows the threads cover at a time
    static_assert(NT % PER == 0, "a thread keeps its column");
    const int r0 = threadIdx.x / PER, c = threadIdx.x % PER * 8;
    const bool col_on = c < n_cols;
    const __nv_bfloat16 *at = src + (col_on ? (size_t)r0 * ld + c : 0);
    dst += (r0 * LD + c) * 2;
#pragma unroll
    for (int k = 0; k < 3; ++k)
#pragma unroll
        for (int r = 0; r < ROWS; r += STEP)
            if (STEP <= ROWS || r0 < ROWS) {
                const bool on = col_on && r0 + r < n_rows;
                cp16_if(dst + (k * ROWS + r) * LD * 2, on ? at + k * plane + (size_t)r * ld : src, on);
            }
}

// acc[i][j] += A B over 16 rows of the contraction: A's fragments are in a[i][plane], B's planes in shared memory at b (row
// k, column 0 of the warp's 8 NT columns), rows LD elements and planes `plane` elements apart. acc[i][j]: rows lane / 4 and 8
// further down of the i-th sixteen, columns 8 j + 2 (lane % 4) and the next. Of the nine products of the parts the three
// below 2^-24 of the whole are left out.
template <int MT, int NT, int LD>
__device__ __forceinline__ void product16(const uint32_t (&a)[MT][3][4], uint32_t b, int plane, float (&acc)[MT][NT][4])
{
    const int lane = threadIdx.x % 32;
    const uint32_t at = b + ((lane & 15) * LD + (lane >> 4) * 8) * 2;
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
        uint32_t w[3][4];
#pragma unroll
        for (int k = 0; k < 3; ++k) ldsm4_t(at + (k * plane + j * 8) * 2, w[k]);
#pragma unroll
        for (int sum = 2; sum >= 0; --sum)                   // small products first
#pragma unroll
            for (int x = 0; x <= sum; ++x)
#pragma unroll
                for (int i = 0; i < MT; ++i) {
                    mma_bf16(acc[i][j], a[i][x], w[sum - x][0], w[sum - x][1]);
                    mma_bf16(acc[i][j + 1], a[i][x], w[sum - x][2], w[sum - x][3]);
                }
    }
}

// The states before every chunk and after the last: a block walks the chunks with 16 MW channels x 64 columns of one head's
// state in registers (MW warps by 4 / MW), the operands of the next chunk in flight.
constexpr int SV = 64, S_THREADS = 128, S_VLD = SV + 8;
template <int MW> struct States { static constexpr int SD = 16 * MW, NT = 2 * MW, STAGES = MW == 1 ? 3 : 2, KLD = SD + 8, TILE = 3 * C * (KLD + S_VLD); };
template <int MW>
__global__ void __launch_bounds__(S_THREADS) gla_states_kernel(const __grid_constant__ b200_gla_args p, int n_chunks)
{
    constexpr int SD = States<MW>::SD, S_NT = States<MW>::NT, S_STAGES = States<MW>::STAGES, S_KLD = States<MW>::KLD, S_TILE = States<MW>::TILE;
    extern __shared__ __align__(16) unsigned char smem[];    // [S_STAGES] x { keys [3][C][S_KLD], values [3][C][S_VLD] }
    const int h = blockIdx.z, d0 = blockIdx.x * SD, j0 = blockIdx.y * SV, tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
    const int d8 = up8(p.dim), d16 = up16(p.dim), v8 = up8(p.vdim), md = warp / (4 / MW) * 16, mj = warp % (4 / MW) * 8 * S_NT;
    const int d = d0 + md + lane / 4, j = j0 + mj + lane % 4 * 2;            // this lane's channels d and d + 8, columns j + 8 k and the next
    const size_t slot = (size_t)p.heads * p.dim * v8;
    const uint32_t base = smem_u32(smem);
    auto fetch = [&](int chunk) {
        const size_t ch = (size_t)chunk * p.heads + h;
        const uint32_t kt = base + (chunk % S_STAGES) * S_TILE * 2;
        fetch_planes<C, SD, S_KLD, S_THREADS>(kt, static_cast<const __nv_bfloat16 *>(p.d_kd) + ch * 3 * C * d16 + d0, (size_t)C * d16, d16, C, d16 - d0);
        fetch_planes<C, SV, S_VLD, S_THREADS>(kt + 3 * C * S_KLD * 2, static_cast<const __nv_bfloat16 *>(p.d_values) + ch * 3 * C * v8 + j0, (size_t)C * v8, v8, C, v8 - j0);
    };
    for (int c = 0; c < S_STAGES - 1; ++c) {
        if (c < n_chunks) fetch(c);
        cp_commit();
    }
    float s[S_NT][4];
#pragma unroll
    for (int k = 0; k < S_NT; ++k)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float2 v = make_float2(0, 0);
            if (p.pos0 > 0 && d + 8 * r < p.dim && j + 8 * k < v8)
                v = *reinterpret_cast<const float2 *>(p.d_state + (size_t)(p.pos0 % p.n_slots) * slot + ((size_t)h * p.dim + d + 8 * r) * v8 + j + 8 * k);
            s[k][2 * r] = v.x; s[k][2 * r + 1] = v.y;
        }
    float next[2];                                           // log2 decays, a chunk ahead
    auto fetch_decay = [&](int c) {
#pragma unroll
        for (int r = 0; r < 2; ++r) next[r] = c < n_chunks && d + 8 * r < d8 ? p.d_decay[((size_t)c * p.heads + h) * d8 + d + 8 * r] : 0.0f;
    };
    fetch_decay(0);
    for (int c = 0; c < n_chunks; ++c) {
        if (c > 0 || p.pos0 > 0) {                           // (nothing reads a state of zeros)
            __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.d_chunk_state) + ((size_t)c * p.heads + h) * 3 * p.dim * v8 + (size_t)d * v8 + j;
#pragma unroll
            for (int k = 0; k < S_NT; ++k)
#pragma unroll
                for (int r = 0; r < 2; ++r)
                    if (d + 8 * r < p.dim && j + 8 * k < v8)
                        put_split2(out + 8 * r * v8 + 8 * k, (size_t)p.dim * v8, s[k][2 * r], s[k][2 * r + 1]);
        }
        const Decay a[2] = {decay_of(next[0] * 0.6931471805599453f), decay_of(next[1] * 0.6931471805599453f)};
        fetch_decay(c + 1);
        cp_wait<S_STAGES - 2>();
        __syncthreads();                                     // this chunk's tiles are there; everybody is done with the previous one's
        if (c + S_STAGES - 1 < n_chunks) fetch(c + S_STAGES - 1);
        cp_commit();
        const uint32_t kt = base + (c % S_STAGES) * S_TILE * 2, vt = kt + 3 * C * S_KLD * 2;
        float u[1][S_NT][4] = {};
        // A[m = channel][k = token] out of rows of tokens: transposed on load, (k 0-7, m 0-7), (k 0-7, m 8-15), (k 8-15, m 0-7), ...
        const uint32_t ka = kt + (((lane & 7) + ((lane >> 4) << 3)) * S_KLD + md + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
        for (int k = 0; k < C; k += 16) {
            uint32_t f[1][3][4];
#pragma unroll
            for (int x = 0; x < 3; ++x) ldsm4_t(ka + (x * C * S_KLD + k * S_KLD) * 2, f[0][x]);
            product16<1, S_NT, S_VLD>(f, vt + (k * S_VLD + mj) * 2, C * S_VLD, u);
        }
#pragma unroll
        for (int k = 0; k < S_NT; ++k)
#pragma unroll
            for (int r = 0; r < 4; ++r) s[k][r] = decayed(s[k][r], a[r >> 1], u[0][k][r]);
    }
    float *out = p.d_state + (size_t)((p.pos0 + p.n_rows) % p.n_slots) * slot;
#pragma unroll
    for (int k = 0; k < S_NT; ++k)
#pragma unroll
        for (int r = 0; r < 2; ++r)
            if (d + 8 * r < p.dim && j + 8 * k < v8)
                *reinterpret_cast<float2 *>(out + ((size_t)h * p.dim + d + 8 * r) * v8 + j + 8 * k) = make_float2(s[k][2 * r], s[k][2 * r + 1]);
}

// Outputs of a chunk, 64 tokens x 64 TN columns per block: decayed queries times the state before the chunk, scores times
// values, 16 rows of the contraction at a time. FUSED: the columns are the whole head, so the norm and the gate follow here.
constexpr int KB = 16, O_STAGES = 4, O_ALD = KB + 8;
template <int TN> constexpr size_t out_tile_bytes = (size_t)3 * (C * O_ALD + KB * (64 * TN + 8)) * 2;
template <int TN, bool FUSED, typename T>
__global__ void __launch_bounds__(THREADS) gla_out_kernel(const __grid_constant__ b200_gla_args p)
{
    constexpr int BW = 64 * TN, BLD = BW + 8, MT = TN, WN = BW / 32;         // warps: 4 / TN by WN
    extern __shared__ __align__(16) unsigned char smem[];    // [O_STAGES] x { A [3][C][O_ALD], B [3][KB][BLD] }
    __shared__ float row_ss[C][WN];
    const int chunk = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * BW;
    const int tid = threadIdx.x, warp = tid / 32, lane = tid % 32, mt = warp / WN * 16 * MT, mj = warp % WN * 32;
    const int d16 = up16(p.dim), v8 = up8(p.vdim), m0 = chunk * C, n = min(C, p.n_rows - m0);
    const size_t ch = (size_t)chunk * p.heads + h;
    const __nv_bfloat16 *S = static_cast<const __nv_bfloat16 *>(p.d_chunk_state) + ch * 3 * p.dim * v8 + j0;
    const __nv_bfloat16 *V = static_cast<const __nv_bfloat16 *>(p.d_values) + ch * 3 * C * v8 + j0;
    const __nv_bfloat16 *Q = static_cast<const __nv_bfloat16 *>(p.d_qd) + ch * 3 * C * d16, *A = static_cast<const __nv_bfloat16 *>(p.d_scores) + ch * 3 * C * C;
    const int steps_s = chunk == 0 && p.pos0 == 0 ? 0 : (p.dim + KB - 1) / KB, steps = steps_s + C / KB;
    const uint32_t base = smem_u32(smem);
    auto fetch = [&](int i) {
        const uint32_t at = base + (i % O_STAGES) * (uint32_t)out_tile_bytes<TN>, bt = at + 3 * C * O_ALD * 2;
        if (i < steps_s) {
            fetch_planes<C, KB, O_ALD, THREADS>(at, Q + i * KB, (size_t)C * d16, d16, C, d16 - i * KB);
            fetch_planes<KB, BW, BLD, THREADS>(bt, S + (size_t)i * KB * v8, (size_t)p.dim * v8, v8, p.dim - i * KB, v8 - j0);
        } else {
            const int k0 = (i - steps_s) * KB;
            fetch_planes<C, KB, O_ALD, THREADS>(at, A + k0, (size_t)C * C, C, C, KB);
            fetch_planes<KB, BW, BLD, THREADS>(bt, V + (size_t)k0 * v8, (size_t)C * v8, v8, KB, v8 - j0);
        }
    };
    for (int i = 0; i < O_STAGES - 1; ++i) {
        if (i < steps) fetch(i);
        cp_commit();
    }
    float acc[MT][4][4] = {};
    for (int i = 0; i < steps; ++i) {
        cp_wait<O_STAGES - 2>();
        __syncthreads();
        if (i + O_STAGES - 1 < steps) fetch(i + O_STAGES - 1);
        cp_commit();
        const uint32_t at = base + (i % O_STAGES) * (uint32_t)out_tile_bytes<TN>, bt = at + 3 * C * O_ALD * 2;
        const uint32_t aa = at + ((mt + (lane & 15)) * O_ALD + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int k = 0; k < KB; k += 16) {
            uint32_t f[MT][3][4];
#pragma unroll
            for (int r = 0; r < MT; ++r)
#pragma unroll
                for (int x = 0; x < 3; ++x) ldsm4(aa + ((x * C + 16 * r) * O_ALD + k) * 2, f[r][x]);
            product16<MT, 4, BLD>(f, bt + (k * BLD + mj) * 2, KB * BLD, acc);
        }
    }
    // rows of this lane: mt + 16 i + lane / 4 and 8 further down
    if (FUSED) {                                             // columns past vdim are zero
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                float ss = 0.0f;
#pragma unroll
                for (int j = 0; j < 4; ++j) ss = fmaf(acc[i][j][2 * r], acc[i][j][2 * r], fmaf(acc[i][j][2 * r + 1], acc[i][j][2 * r + 1], ss));
                ss += __shfl_xor_sync(0xffffffffu, ss, 1);
                ss += __shfl_xor_sync(0xffffffffu, ss, 2);
                if (lane % 4 == 0) row_ss[mt + 16 * i + lane / 4 + 8 * r][warp % WN] = ss;
            }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = mt + 16 * i + lane / 4 + 8 * r;
            if (t >= n) continue;
            const size_t m = (size_t)m0 + t;
            const int col = j0 + mj + lane % 4 * 2;
            float inv = 1.0f, gate[4][2];
            if (FUSED) {
                const float *src = p.d_gate + m * p.proj_ld + (size_t)h * p.vdim + col;
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int e = 0; e < 2; ++e) gate[j][e] = col + 8 * j + e < p.vdim ? __ldg(src + 8 * j + e) : 0.0f;
                float ss = 0.0f;
#pragma unroll
                for (int w = 0; w < WN; ++w) ss += row_ss[t][w];
                inv = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int c = col + 8 * j + e;
                    if (c >= p.vdim) continue;
                    const float o = acc[i][j][2 * r + e];
                    if (FUSED) static_cast<T *>(p.d_out_rows)[m * p.out_ld + (size_t)h * p.vdim + c] = (T)(__ldg(p.d_norm_gamma + c) * (o * inv) * silu_f32(gate[j][e]));
                    else p.d_o[m * p.heads * p.vdim + (size_t)h * p.vdim + c] = o;
                }
        }
}

// Norm and gate of heads wider than a block of gla_out: a warp per token and head.
template <typename T>
__global__ void __launch_bounds__(THREADS) gla_gate_kernel(const __grid_constant__ b200_gla_args p)
{
    const int lane = threadIdx.x & 31;
    const size_t w = (size_t)blockIdx.x * (THREADS / 32) + (threadIdx.x >> 5);
    if (w >= (size_t)p.n_rows * p.heads) return;
    const size_t m = w / p.heads, h = w % p.heads;
    const float *o = p.d_o + (m * p.heads + h) * p.vdim, *gate = p.d_gate + m * p.proj_ld + h * p.vdim;
    float ss = 0.0f;
    for (int j = lane; j < p.vdim; j += 32) ss = fmaf(o[j], o[j], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    T *out = static_cast<T *>(p.d_out_rows) + m * p.out_ld + h * p.vdim;
    for (int j = lane; j < p.vdim; j += 32) out[j] = (T)(p.d_norm_gamma[j] * (o[j] * inv) * silu_f32(gate[j]));
}

// ------------------------------------------------------------------------------------------------ host side

bool shape_ok(const b200_gla_args *a)
{
    return a && a->heads > 0 && a->dim > 0 && a->vdim > 0 && a->rank > 0 && a->n_slots > 1 && a->tau > 0.0f && a->d_q && a->d_k && a->d_v &&
           a->d_gate && a->d_f && a->d_a2 && a->d_a2_bias && a->d_norm_gamma && a->d_state;
}

template <typename K>
int allow_smem(K kern, size_t smem)
{
    if (smem > 220 * 1024) return B200_E_TOOLARGE;
    return smem > 48 * 1024 ? (int)cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : 0;
}

template <int MW>
int walk_states(const b200_gla_args &a, int n_chunks, cudaStream_t st)
{
    using S = States<MW>;
    const size_t smem = (size_t)S::STAGES * S::TILE * 2;
    const int rc = allow_smem(gla_states_kernel<MW>, smem);
    if (rc) return rc;
    gla_states_kernel<MW><<<dim3((a.dim + S::SD - 1) / S::SD, (a.vdim + SV - 1) / SV, a.heads), S_THREADS, smem, st>>>(a, n_chunks);
    ++g_b200_launches;
    return (int)cudaGetLastError();
}

template <int TN, typename T>
int out_rows(const b200_gla_args &a, int n_chunks, cudaStream_t st)
{
    const int tiles = (a.vdim + 64 * TN - 1) / (64 * TN);
    const size_t smem = O_STAGES * out_tile_bytes<TN>;
    const dim3 grid(n_chunks, a.heads, tiles);
    int rc;
    if (tiles == 1) {
        if ((rc = allow_smem(gla_out_kernel<TN, true, T>, smem)) != 0) return rc;
        gla_out_kernel<TN, true, T><<<grid, THREADS, smem, st>>>(a);
        ++g_b200_launches;
        return (int)cudaGetLastError();
    }
    if ((rc = allow_smem(gla_out_kernel<TN, false, T>, smem)) != 0) return rc;
    gla_out_kernel<TN, false, T><<<grid, THREADS, smem, st>>>(a);
    const size_t warps = (size_t)a.n_rows * a.heads;
    gla_gate_kernel<T><<<(unsigned)((warps + 7) / 8), THREADS, 0, st>>>(a);
    g_b200_launches += 2;
    return (int)cudaGetLastError();
}

}  // namespace

extern "C" int b200_gla_decode(const b200_gla_args *a, void *stream)
{
    if (!shape_ok(a) || !a->d_out || !a->d_pos || ((uintptr_t)a->d_f & 15)) return B200_E_BADARG;
    const int quads = up8(a->vdim) / 4;
    int cl = 1;                                              // four quads a block or more, and no more blocks than SMs
    while (cl < MAX_CLUSTER && quads > 4 * cl && a->heads * cl * 2 <= 148) cl <<= 1;
    while (cl < MAX_CLUSTER && (quads + cl - 1) / cl > 32) cl <<= 1;
    int vg = 1;
    while (vg < (quads + cl - 1) / cl) vg <<= 1;
    if (vg > 32) return B200_E_TOOLARGE;
    const int R4 = up4(a->rank);
    const size_t smem = ((size_t)4 * up4(a->dim) + THREADS / 32 * 4 * vg + (size_t)a->dim * ((R4 / 4) | 1) * 4) * 4;
    const int rc = allow_smem(gla_decode_kernel, smem);
    if (rc) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a->heads * cl);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = (cudaStream_t)stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cl; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a->use_pdl ? 2 : 1;
    ++g_b200_launches;
    return (int)cudaLaunchKernelEx(&cfg, gla_decode_kernel, *a, vg, cl);
}

extern "C" int b200_gla_rows(const b200_gla_args *ap, void *stream)
{
    if (!shape_ok(ap) || ap->n_rows < 1 || ap->pos0 < 0 || ap->proj_ld < 1 || !ap->d_qd || !ap->d_kd || !ap->d_values || !ap->d_decay || !ap->d_scores ||
        !ap->d_chunk_state || !ap->d_out_rows || (ap->vdim > 128 && !ap->d_o) || ap->out_ld < (long long)ap->heads * ap->vdim ||
        (ap->wtype != B200_WT_BF16 && ap->wtype != B200_WT_F32))
        return B200_E_BADARG;
    const b200_gla_args &a = *ap;
    cudaStream_t st = (cudaStream_t)stream;
    const int n_chunks = (a.n_rows + C - 1) / C, R4 = up4(a.rank);
    const size_t prep = ((size_t)C * R4 + (size_t)(5 * C + 96) * RS + (size_t)DT * ((R4 / 4) | 1) * 4) * 4;
    int rc = allow_smem(gla_prep_kernel, prep);
    if (rc) return rc;
    gla_prep_kernel<<<dim3(n_chunks, a.heads), THREADS, prep, st>>>(a);
    ++g_b200_launches;
    // the larger tile where it still gives every SM a block
    const bool large = (long long)a.heads * ((a.dim + 31) / 32) * ((a.vdim + SV - 1) / SV) >= 128;
    if ((rc = large ? walk_states<2>(a, n_chunks, st) : walk_states<1>(a, n_chunks, st)) != 0) return rc;
    if (a.wtype == B200_WT_BF16) return a.vdim <= 64 ? out_rows<1, __nv_bfloat16>(a, n_chunks, st) : out_rows<2, __nv_bfloat16>(a, n_chunks, st);
    return a.vdim <= 64 ? out_rows<1, float>(a, n_chunks, st) : out_rows<2, float>(a, n_chunks, st);
}
