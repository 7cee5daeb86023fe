// Gated linear attention (sm_100a): per head a state S [dim][vdim] that decays by a factor per key channel and takes in
// one outer product per token, everything from the projections on in fp32.
//
// Decode, one launch: a cluster of blocks per head, each block a slice of the columns. The state slice and the weights
// of the decay are fetched before the kernel waits for its predecessor; the norm over a head's result is a sum across
// the cluster through distributed shared memory.
//
// Prompt portions: chunks of 64 tokens in parallel. With c_t the running sum of the log decays inside a chunk,
//   o_t = (q_t exp(c_t)) S_in + sum over s <= t of (sum over channels q_t k_s exp(c_t - c_s)) v_s
//   S_out = exp(c_end) S_in + sum over s of (k_s exp(c_end - c_s)) v_s^T
// gla_prep forms the decayed queries and keys and the score matrix, gla_chunk_state every chunk's own sum,
// gla_scan joins the chunks, gla_out forms the outputs. Every exponent that is taken is <= 0: inside sixteen tokens the
// differences c_t - c_s are exponentiated pair by pair, across sixteens through the value of c between the two.
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

// One block per chunk and head. Shared: f [C][R4], then [C][RS] each: c (running log decay), q, k, q from the start of
// its sixteen; and k up to the starts of the second, third and fourth sixteen, [16 + 32 + 48][RS].
__global__ void __launch_bounds__(THREADS) gla_prep_kernel(const __grid_constant__ b200_gla_args p)
{
    extern __shared__ __align__(16) float sh[];
    __shared__ float tot[8][DT];
    const int R4 = up4(p.rank), d8 = up8(p.dim), tid = threadIdx.x;
    float *fs = sh, *cs = fs + C * R4, *qs = cs + C * RS, *ks = qs + C * RS, *qh = ks + C * RS, *kh = qh + C * RS, *ws = kh + 96 * RS;
    const int chunk = blockIdx.x, h = blockIdx.y, m0 = chunk * C, n = min(C, p.n_rows - m0);
    const int w16 = (R4 / 4) | 1;
    for (int e = tid; e < C * R4; e += THREADS) {
        const int t = e / R4, r = e % R4;
        fs[e] = t < n && r < p.rank ? p.d_f[(size_t)(m0 + t) * p.proj_ld + r] : 0.0f;
    }
    const int ti = tid / SUB, si = tid % SUB;
    float acc[10];                                           // (i, j) of the lower triangle of sixteens, j <= i
#pragma unroll
    for (int x = 0; x < 10; ++x) acc[x] = 0.0f;

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
                q[i] = on && t < n ? p.d_q[(size_t)(m0 + t) * p.proj_ld + at] * p.q_scale : 0.0f;
                k[i] = on && t < n ? p.d_k[(size_t)(m0 + t) * p.proj_ld + at] : 0.0f;
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
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (on && tg * 8 + i < n) run += log_logistic(c[i]) / p.tau;
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
            if (d0 + d < d8) {
                const size_t at = ((size_t)m0 + t) * p.heads * d8 + (size_t)h * d8 + d0 + d;
                p.d_qd[at] = q[i] * expf(c[i]);
                p.d_kd[at] = k[i] * expf(end - c[i]);
            }
        }
        if (tg == 0 && d0 + d < d8) p.d_decay[((size_t)chunk * p.heads + h) * d8 + d0 + d] = end;
        __syncthreads();
        // references: c just before each sixteen
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            const int t = tg * 8 + i, u = t / SUB;
            if (u > 0) qh[t * RS + d] = q[i] * expf(c[i] - cs[(u * SUB - 1) * RS + d]);
#pragma unroll
            for (int v = 1; v < 4; ++v)
                if (u < v) kh[(v * (v - 1) * SUB / 2 + t) * RS + d] = k[i] * expf(cs[(v * SUB - 1) * RS + d] - c[i]);
        }
        __syncthreads();
#pragma unroll 2
        for (int x = 0; x < DT; x += 4) {
#pragma unroll
            for (int i = 0, at = 0; i < 4; ++i) {
                if (i > 0) {
                    const float4 a = *reinterpret_cast<const float4 *>(qh + (i * SUB + ti) * RS + x);
#pragma unroll
                    for (int j = 0; j < i; ++j, ++at)
                        acc[at] = dot4(a, *reinterpret_cast<const float4 *>(kh + (i * (i - 1) * SUB / 2 + j * SUB + si) * RS + x), acc[at]);
                }
                const float4 a = *reinterpret_cast<const float4 *>(qs + (i * SUB + ti) * RS + x), b = *reinterpret_cast<const float4 *>(ks + (i * SUB + si) * RS + x);
                const float4 e = *reinterpret_cast<const float4 *>(cs + (i * SUB + ti) * RS + x), f = *reinterpret_cast<const float4 *>(cs + (i * SUB + si) * RS + x);
                if (si <= ti) {
                    const float4 w = make_float4(__expf(e.x - f.x), __expf(e.y - f.y), __expf(e.z - f.z), __expf(e.w - f.w));
                    acc[at] = dot4(make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w), w, acc[at]);
                }
                ++at;
            }
        }
    }
    float *out = p.d_scores + ((size_t)chunk * p.heads + h) * C * C;
#pragma unroll
    for (int i = 0, at = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j <= i; ++j, ++at) out[(i * SUB + ti) * C + j * SUB + si] = acc[at];
}

// Tile product: acc[4][4 * TN] += A[k][m] B[k][n] over kn rows of shared tiles, thread (ty, tx): rows 4 ty.., columns 4 tx + 64 g..
template <int TN>
__device__ __forceinline__ void tile_product(const float *A, int lda, const float *B, int ldb, int kn, int ty, int tx, float (&acc)[4][4 * TN])
{
#pragma unroll 4
    for (int k = 0; k < kn; ++k) {
        const float4 a4 = *reinterpret_cast<const float4 *>(A + k * lda + 4 * ty);
        const float a[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
        for (int g = 0; g < TN; ++g) {
            const float4 b = *reinterpret_cast<const float4 *>(B + k * ldb + 64 * g + 4 * tx);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                acc[i][4 * g] = fmaf(a[i], b.x, acc[i][4 * g]); acc[i][4 * g + 1] = fmaf(a[i], b.y, acc[i][4 * g + 1]);
                acc[i][4 * g + 2] = fmaf(a[i], b.z, acc[i][4 * g + 2]); acc[i][4 * g + 3] = fmaf(a[i], b.w, acc[i][4 * g + 3]);
            }
        }
    }
}

// A chunk's own sum: 64 channels x 64 TN columns per block.
template <int TN>
__global__ void __launch_bounds__(THREADS) gla_chunk_state_kernel(const __grid_constant__ b200_gla_args p, int vtiles)
{
    __shared__ __align__(16) float ks[C][64 + 4], vs[C / 2][64 * TN + 4];
    const int chunk = blockIdx.x, h = blockIdx.y, d0 = blockIdx.z / vtiles * 64, j0 = blockIdx.z % vtiles * 64 * TN;
    const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16, d8 = up8(p.dim), v8 = up8(p.vdim), m0 = chunk * C, n = min(C, p.n_rows - m0);
    for (int e = tid; e < C * 16; e += THREADS) {
        const int t = e / 16, d = e % 16 * 4;
        *reinterpret_cast<float4 *>(&ks[t][d]) = d0 + d < d8 ? *reinterpret_cast<const float4 *>(p.d_kd + ((size_t)m0 + t) * p.heads * d8 + (size_t)h * d8 + d0 + d)
                                                            : make_float4(0, 0, 0, 0);
    }
    float acc[4][4 * TN];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4 * TN; ++j) acc[i][j] = 0.0f;
    for (int t0 = 0; t0 < C; t0 += C / 2) {
        __syncthreads();
        for (int e = tid; e < C / 2 * 64 * TN; e += THREADS) {
            const int t = e / (64 * TN), j = e % (64 * TN);
            vs[t][j] = t0 + t < n && j0 + j < p.vdim ? p.d_v[(size_t)(m0 + t0 + t) * p.proj_ld + (size_t)h * p.vdim + j0 + j] : 0.0f;
        }
        __syncthreads();
        tile_product<TN>(&ks[t0][0], 64 + 4, &vs[0][0], 64 * TN + 4, C / 2, ty, tx, acc);
    }
    float *out = p.d_chunk_state + ((size_t)chunk * p.heads + h) * p.dim * v8;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int g = 0; g < TN; ++g) {
            const int d = d0 + 4 * ty + i, j = j0 + 64 * g + 4 * tx;
            if (d < p.dim && j < v8)
                *reinterpret_cast<float4 *>(out + (size_t)d * v8 + j) = make_float4(acc[i][4 * g], acc[i][4 * g + 1], acc[i][4 * g + 2], acc[i][4 * g + 3]);
        }
}

// Replaces every chunk's own sum by the state before it; the state after the last one goes to its slot. A thread: one quad.
__global__ void __launch_bounds__(THREADS) gla_scan_kernel(const __grid_constant__ b200_gla_args p, int n_chunks)
{
    constexpr int AHEAD = 8;
    const int v8 = up8(p.vdim), d8 = up8(p.dim), quads = v8 / 4;
    const size_t e = (size_t)blockIdx.x * THREADS + threadIdx.x, total = (size_t)p.heads * p.dim * quads, per = total * 4;
    if (e >= total) return;
    const size_t row = e / quads;                            // head * dim + channel
    const size_t ch = row / p.dim * d8 + row % p.dim;
    float4 s = make_float4(0, 0, 0, 0);
    if (p.pos0 > 0) s = *reinterpret_cast<const float4 *>(p.d_state + (size_t)(p.pos0 % p.n_slots) * per + e * 4);
    for (int c0 = 0; c0 < n_chunks; c0 += AHEAD) {
        float4 u[AHEAD];
        Decay g[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (c0 + i < n_chunks) {
                u[i] = *reinterpret_cast<const float4 *>(p.d_chunk_state + (size_t)(c0 + i) * per + e * 4);
                g[i] = decay_of(p.d_decay[(size_t)(c0 + i) * p.heads * d8 + ch]);
            }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (c0 + i < n_chunks) {
                *reinterpret_cast<float4 *>(p.d_chunk_state + (size_t)(c0 + i) * per + e * 4) = s;
                s.x = decayed(s.x, g[i], u[i].x); s.y = decayed(s.y, g[i], u[i].y); s.z = decayed(s.z, g[i], u[i].z); s.w = decayed(s.w, g[i], u[i].w);
            }
    }
    *reinterpret_cast<float4 *>(p.d_state + (size_t)((p.pos0 + p.n_rows) % p.n_slots) * per + e * 4) = s;
}

// Outputs of a chunk, 64 tokens x 64 TN columns per block: decayed queries times the state before the chunk, scores times
// values. FUSED: the columns are the whole head, so the norm and the gate follow here.
template <int TN, bool FUSED, typename T>
__global__ void __launch_bounds__(THREADS) gla_out_kernel(const __grid_constant__ b200_gla_args p)
{
    constexpr int KB = 32, BW = 64 * TN + 4;
    __shared__ __align__(16) float as[KB][C + 4], bs[KB][BW];
    const int chunk = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * 64 * TN;
    const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16, d8 = up8(p.dim), v8 = up8(p.vdim), m0 = chunk * C, n = min(C, p.n_rows - m0);
    const float *S = p.d_chunk_state + ((size_t)chunk * p.heads + h) * p.dim * v8;
    const float *A = p.d_scores + ((size_t)chunk * p.heads + h) * C * C;
    float acc[4][4 * TN];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4 * TN; ++j) acc[i][j] = 0.0f;
    for (int k0 = 0; k0 < p.dim; k0 += KB) {
        __syncthreads();
        for (int e = tid; e < C * KB; e += THREADS) {        // lanes over channels: coalesced; rows of `as` 4 banks apart
            const int t = e / KB, k = e % KB;
            as[k][t] = k0 + k < d8 ? p.d_qd[((size_t)m0 + t) * p.heads * d8 + (size_t)h * d8 + k0 + k] : 0.0f;
        }
        for (int e = tid; e < KB * 16 * TN; e += THREADS) {
            const int k = e / (16 * TN), j = e % (16 * TN) * 4;
            *reinterpret_cast<float4 *>(&bs[k][j]) = k0 + k < p.dim && j0 + j < v8 ? *reinterpret_cast<const float4 *>(S + (size_t)(k0 + k) * v8 + j0 + j)
                                                                                  : make_float4(0, 0, 0, 0);
        }
        __syncthreads();
        tile_product<TN>(&as[0][0], C + 4, &bs[0][0], BW, KB, ty, tx, acc);
    }
    for (int k0 = 0; k0 < C; k0 += KB) {
        __syncthreads();
        for (int e = tid; e < C * KB; e += THREADS) {
            const int t = e / KB, k = e % KB;
            as[k][t] = (k0 + k) / SUB <= t / SUB ? A[t * C + k0 + k] : 0.0f;       // sixteens above the diagonal are not stored
        }
        for (int e = tid; e < KB * 64 * TN; e += THREADS) {
            const int k = e / (64 * TN), j = e % (64 * TN);
            bs[k][j] = k0 + k < n && j0 + j < p.vdim ? p.d_v[(size_t)(m0 + k0 + k) * p.proj_ld + (size_t)h * p.vdim + j0 + j] : 0.0f;
        }
        __syncthreads();
        tile_product<TN>(&as[0][0], C + 4, &bs[0][0], BW, KB, ty, tx, acc);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        float inv = 1.0f;
        if (FUSED) {
            float ss = 0.0f;                                 // columns past vdim are zero
#pragma unroll
            for (int j = 0; j < 4 * TN; ++j) ss = fmaf(acc[i][j], acc[i][j], ss);
#pragma unroll
            for (int o = 1; o < 16; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            inv = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
        }
        if (t >= n) continue;
        const size_t m = (size_t)m0 + t;
#pragma unroll
        for (int g = 0; g < TN; ++g)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int col = j0 + 64 * g + 4 * tx + j;
                if (col >= p.vdim) continue;
                if (FUSED)
                    static_cast<T *>(p.d_out_rows)[m * p.out_ld + (size_t)h * p.vdim + col] =
                        (T)(p.d_norm_gamma[col] * (acc[i][4 * g + j] * inv) * silu_f32(p.d_gate[m * p.proj_ld + (size_t)h * p.vdim + col]));
                else p.d_o[m * p.heads * p.vdim + (size_t)h * p.vdim + col] = acc[i][4 * g + j];
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

template <int TN, typename T>
int out_rows(const b200_gla_args &a, int n_chunks, cudaStream_t st)
{
    const int tiles = (a.vdim + 64 * TN - 1) / (64 * TN);
    const dim3 grid(n_chunks, a.heads, tiles);
    if (tiles == 1) {
        gla_out_kernel<TN, true, T><<<grid, THREADS, 0, st>>>(a);
        ++g_b200_launches;
        return (int)cudaGetLastError();
    }
    gla_out_kernel<TN, false, T><<<grid, THREADS, 0, st>>>(a);
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
    if (!shape_ok(ap) || ap->n_rows < 1 || ap->pos0 < 0 || ap->proj_ld < 1 || !ap->d_qd || !ap->d_kd || !ap->d_decay || !ap->d_scores ||
        !ap->d_chunk_state || !ap->d_out_rows || (ap->vdim > 128 && !ap->d_o) || ap->out_ld < (long long)ap->heads * ap->vdim ||
        (ap->wtype != B200_WT_BF16 && ap->wtype != B200_WT_F32))
        return B200_E_BADARG;
    const b200_gla_args &a = *ap;
    cudaStream_t st = (cudaStream_t)stream;
    const int n_chunks = (a.n_rows + C - 1) / C, R4 = up4(a.rank), v8 = up8(a.vdim);
    const size_t smem = ((size_t)C * R4 + (size_t)(4 * C + 96) * RS + (size_t)DT * ((R4 / 4) | 1) * 4) * 4;
    int rc = allow_smem(gla_prep_kernel, smem);
    if (rc) return rc;
    gla_prep_kernel<<<dim3(n_chunks, a.heads), THREADS, smem, st>>>(a);
    const int dtiles = (a.dim + 63) / 64;
    if (a.vdim <= 64) gla_chunk_state_kernel<1><<<dim3(n_chunks, a.heads, dtiles), THREADS, 0, st>>>(a, 1);
    else {
        const int vt = (a.vdim + 127) / 128;
        gla_chunk_state_kernel<2><<<dim3(n_chunks, a.heads, dtiles * vt), THREADS, 0, st>>>(a, vt);
    }
    const size_t quads = (size_t)a.heads * a.dim * (v8 / 4);
    gla_scan_kernel<<<(unsigned)((quads + THREADS - 1) / THREADS), THREADS, 0, st>>>(a, n_chunks);
    g_b200_launches += 3;
    if ((rc = (int)cudaGetLastError()) != 0) return rc;
    if (a.wtype == B200_WT_BF16) return a.vdim <= 64 ? out_rows<1, __nv_bfloat16>(a, n_chunks, st) : out_rows<2, __nv_bfloat16>(a, n_chunks, st);
    return a.vdim <= 64 ? out_rows<1, float>(a, n_chunks, st) : out_rows<2, float>(a, n_chunks, st);
}
