// Fused weight-streaming matrix-vector product for batch-1 decode (sm_100a).
//
// One block per SM slot owns a contiguous range of rows. A producer warp
// streams that range through a shared-memory ring with bulk asynchronous
// copies (TMA, cp.async.bulk + mbarrier): rows of a packed matrix are
// contiguous, so one copy instruction moves a whole stage (RB rows, 16-24 KB)
// and the ring keeps ~100 KB per block in flight without holding registers.
// Consumer threads own fixed 16-byte column slices (16 int8 quants or 8
// halves) of every row, so their slice of the input vector stays in registers
// for the whole kernel; consumer groups take stages round-robin, finish the RB
// rows of a stage with one transposing shuffle reduction per warp plus a
// fixed-order sum over the group's warps (reproducible run to run).
//
// Launched with programmatic dependent launch, a block of the NEXT kernel in
// the stream starts as soon as an SM has room for it (with the default 192 KB
// ring that is when a block of this kernel has left), fills its own ring with
// weights and only then waits for its input.
//
// The math is the reference's q8_matvec / f16_matvec
// (shaders/q8_kernels.metal:10-42, 97-127): fp32 activations, integer quants
// converted to fp32, fp32 multiply-accumulate, partial block sums scaled by
// the binary16 block scale. BF16 and F32 weights have no counterpart there. Input assembly and the epilogues fold in rms_norm
// (:133-157), residual_add (:369-375), silu_mul / gelu_mul (:337-363), the
// embedding copy (src/nn/fast_inference.c:386-392) and argmax (:469-476).
//
// This header holds the kernel and its launchers; matvec.cu instantiates them for Q8_0 and F16 weights, matvec_ext.cu
// and matvec_streams.cu for BF16 and F32 (translation units of their own: they compile side by side).
#pragma once
#include "stream_core.cuh"
#include "../../include/llmb200_kernels.h"

extern unsigned long long g_b200_launches;

namespace b200_mv {

struct Geometry {
    int T;              // threads per consumer group (a multiple of 32)
    int NG;             // consumer groups
    int nstage;         // ring slots
    unsigned slot_bytes;  // bytes per slot (RB rows, rounded up to 128)
    int share_x;        // 1: group 0 assembles the input vector and hands it to the other groups through shared memory
};

// blockDim.x = NG*T consumers + 32 producer threads.
// RMS norm of the vector a group of T threads holds, `groups` equal consecutive parts of its first `dim` elements
// each by its own mean square. In place; one part after the other, so the sums are in a fixed order.
template <int SPT, int E>
__device__ __forceinline__ void norm_parts(float (&x)[SPT][E], const int (&col)[SPT], const float (&gamma)[SPT][E], int dim,
                                           int groups, float eps, float *gred, int bar_id, int T, int t)
{
    const int len = dim / groups;
    for (int k = 0; k < groups; ++k) {
        const int lo = k * len, hi = lo + len;
        float ss = 0.0f;
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e)
                if (col[s] + e >= lo && col[s] + e < hi) ss = fmaf(x[s][e], x[s][e], ss);
        ss = group_sum(ss, gred, bar_id, T, t);
        const float inv = 1.0f / sqrtf(ss / (float)len + eps);
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e)
                if (col[s] + e >= lo && col[s] + e < hi) x[s][e] = gamma[s][e] * (x[s][e] * inv);
    }
}

// Layer norm (mean taken off, variance of the deviations, weight and bias) of the first `dim` elements, in place; the
// columns past them hold zeros before and after (their weight and bias are zero).
template <int SPT, int E>
__device__ __forceinline__ void layer_norm(float (&x)[SPT][E], const int (&col)[SPT], const float (&gamma)[SPT][E],
                                           const float (&beta)[SPT][E], int dim, float eps, float *gred, int bar_id, int T, int t)
{
    float sum = 0.0f;
#pragma unroll
    for (int s = 0; s < SPT; ++s)
#pragma unroll
        for (int e = 0; e < E; ++e) sum += x[s][e];
    const float mean = group_sum(sum, gred, bar_id, T, t) / (float)dim;
    float ss = 0.0f;
#pragma unroll
    for (int s = 0; s < SPT; ++s)
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (col[s] + e < dim) { x[s][e] -= mean; ss = fmaf(x[s][e], x[s][e], ss); }
    ss = group_sum(ss, gred, bar_id, T, t);
    const float inv = 1.0f / sqrtf(ss / (float)dim + eps);
#pragma unroll
    for (int s = 0; s < SPT; ++s)
#pragma unroll
        for (int e = 0; e < E; ++e) x[s][e] = fmaf(gamma[s][e], x[s][e] * inv, beta[s][e]);
}

template <int SPT, int E>
__device__ __forceinline__ void load_slices(float (&v)[SPT][E], const float *src, const int (&col)[SPT], const bool (&on)[SPT])
{
#pragma unroll
    for (int s = 0; s < SPT; ++s)
#pragma unroll
        for (int e = 0; e < E; e += 4) {
            const float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(src + col[s] + e) : make_float4(0, 0, 0, 0);
            v[s][e] = v4.x; v[s][e + 1] = v4.y; v[s][e + 2] = v4.z; v[s][e + 3] = v4.w;
        }
}

// Which of the optional parts an instantiation holds (registers decide how well the row loop runs): FAM_PLAIN the parts
// every weight type has, FAM_POST post-norm inputs, gated outputs, depth sums and the logit cap, FAM_STREAMS layer
// norms, learned positions, residual streams and the squared relu.
enum { FAM_PLAIN = 0, FAM_POST = 1, FAM_STREAMS = 2 };

template <int WT, int SPT, int RB, int MAXT, int FAM>
__global__ void __launch_bounds__(MAXT)
matvec_kernel(const __grid_constant__ b200_matvec_args p, const Geometry geo)
{
    constexpr int E = (WT == B200_WT_Q8) ? 16 : (WT == B200_WT_F32) ? 4 : 8;       // elements per 16-byte slice
    constexpr bool EXT = FAM == FAM_POST, STR = FAM == FAM_STREAMS;
    extern __shared__ __align__(128) unsigned char smem_raw[];
    const int T = geo.T, NG = geo.NG, nstage = geo.nstage, nwg = T >> 5, nC = NG * T;
    unsigned char *ring = smem_raw;
    uint64_t *full = reinterpret_cast<uint64_t *>(ring + (size_t)nstage * geo.slot_bytes);
    uint64_t *empty = full + nstage;
    float *wpart = reinterpret_cast<float *>(empty + nstage);   // [NG][2][nwg][RB]
    float *red = wpart + (size_t)NG * 2 * nwg * RB;             // [NG][32]
    float *am_v = red + NG * 32;                                // [NG*RB]
    int *am_i = reinterpret_cast<int *>(am_v + NG * RB);        // [NG*RB]
    float *xs = reinterpret_cast<float *>(am_i + NG * RB);      // [SPT*T*E] when geo.share_x
    __shared__ int s_last;
    __shared__ float s_conn[STR ? B200_MAX_STREAMS * (B200_MAX_STREAMS + 2) : 1];     // mix, out, next read of the streams

    const int tid = threadIdx.x;
    const int ralign = (p.out_mode == B200_OUT_GLU) ? 2 : 1;
    const long long units = p.rows / ralign;
    const int r0 = (int)(units * blockIdx.x / gridDim.x) * ralign;
    const int r1 = (int)(units * (blockIdx.x + 1) / gridDim.x) * ralign;
    const int nst = (r1 - r0 + RB - 1) / RB;

    if (tid == 0) {
        for (int i = 0; i < nstage; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], T); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();
    // Every thread signals: the next kernel in the stream may be scheduled now and start
    // filling its own ring beside this block.
    pdl_launch_dependents();

    // ---------------- producer warp: weights depend on no earlier kernel ----------------
    if (tid >= nC) {
        if (tid == nC) {
            const unsigned char *wbase = static_cast<const unsigned char *>(p.d_w);
            for (int i = 0; i < nst; ++i) {
                const int slot = i % nstage;
                if (i >= nstage && !mbar_wait(&empty[slot], ((i / nstage) - 1) & 1)) {
                    if (p.d_err) *p.d_err = 2;
                    break;
                }
                const int row0 = r0 + i * RB;
                const int nr = min(RB, r1 - row0);
                const unsigned bytes = (unsigned)nr * (unsigned)p.row_stride;
                mbar_expect_tx(&full[slot], bytes);
                bulk_load(ring + (size_t)slot * geo.slot_bytes, wbase + (long long)row0 * p.row_stride, bytes, &full[slot]);
            }
        } else if constexpr (EXT) {
            // the producer warp's other lanes form the depth sums of this block's rows
            if (p.hist_n > 0) {
                pdl_wait();
                for (int row = r0 + (tid - nC - 1); row < r1; row += 31) {
                    float a = 0.0f;
#pragma unroll 8
                    for (int j = 0; j < p.hist_n; ++j) a = fmaf(p.d_hist_coef[j], p.d_hist[(long long)j * p.hist_stride + row], a);
                    p.d_hist_out[row] = a;
                }
            }
        }
        return;
    }

    // ---------------- consumers ----------------
    const int g = tid / T, t = tid - g * T, lane = t & 31, wg = t >> 5;
    float *gred = red + g * 32;
    int col[SPT];
    bool on[SPT];
#pragma unroll
    for (int s = 0; s < SPT; ++s) { col[s] = (s * T + t) * E; on[s] = col[s] < p.cols; }

    // The norm weights are constants: their round trip is taken before the wait for the previous
    // kernel, not after it.
    float gm[SPT][E];
    const bool pre_gamma = p.d_norm_gamma && (!geo.share_x || g == 0);
    if (pre_gamma) {
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; e += 4) {
                float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(p.d_norm_gamma + col[s] + e) : make_float4(0, 0, 0, 0);
                gm[s][e] = v4.x; gm[s][e + 1] = v4.y; gm[s][e + 2] = v4.z; gm[s][e + 3] = v4.w;
            }
    }

    float gp[EXT ? SPT : 1][E];                  // the same for the norm of a post-norm input
    if constexpr (EXT) {
        if (p.in_mode == B200_IN_POSTNORM && (!geo.share_x || g == 0)) {
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4) {
                    const float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(p.d_slot_norm_gamma + col[s] + e) : make_float4(0, 0, 0, 0);
                    gp[s][e] = v4.x; gp[s][e + 1] = v4.y; gp[s][e + 2] = v4.z; gp[s][e + 3] = v4.w;
                }
        }
    }

    float gb[STR ? SPT : 1][E];                  // bias of a layer norm
    if constexpr (STR) {
        if (pre_gamma && p.d_norm_beta) load_slices<SPT, E>(gb, p.d_norm_beta, col, on);
        if (p.out_mode == B200_OUT_STREAMS && wg == 0) {         // the epilogue warp of every group, same values
            for (int i = lane; i < p.n_streams * (p.n_streams + 2); i += 32) s_conn[i] = p.d_connect[i];
            __syncwarp();
        }
    }

    pdl_wait();

    // Tensor parallel: every rank's partial vector must have landed in `slots`
    // (and, for the first kernel of a token, every rank must be done reading the
    // previous token's slots) before this block goes on.
    if (p.n_wait > 0) {
        if (tid < p.n_wait) {
            const unsigned want = (*p.d_epoch) * (unsigned)p.epoch_mul + (unsigned)p.epoch_add;
            if (!wait_flag_ge(p.d_wait_flags + tid, want, p.spin_limit > 0 ? p.spin_limit : B200_SPIN_LIMIT)) *p.d_err = 1;
        }
        named_barrier(1, nC);
    }

    // ---------------- input assembly ----------------
    // Every SM needs the whole input vector. When it has to be assembled (slot sums, norms), one group
    // per block does it and passes it on through shared memory: the few KB involved are read by all
    // SMs at once, and every extra reader of the same L2 lines queues behind the others.
    float x[SPT][E];
    if (!geo.share_x || g == 0) {
    if (p.in_mode == B200_IN_VEC || (EXT && p.in_mode == B200_IN_POSTNORM)) {
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; e += 4) {
                float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(p.d_in_vec + col[s] + e) : make_float4(0, 0, 0, 0);
                x[s][e] = v4.x; x[s][e + 1] = v4.y; x[s][e + 2] = v4.z; x[s][e + 3] = v4.w;
            }
        if constexpr (EXT) {
            if (p.in_mode == B200_IN_POSTNORM) {
                float mix[SPT][E];                       // fetched before the norm's reductions
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; e += 4) {
                        const float4 v4 = on[s] && p.d_mix_in ? *reinterpret_cast<const float4 *>(p.d_mix_in + col[s] + e) : make_float4(0, 0, 0, 0);
                        mix[s][e] = v4.x; mix[s][e + 1] = v4.y; mix[s][e + 2] = v4.z; mix[s][e + 3] = v4.w;
                    }
                const float coef = p.d_mix_in ? *p.d_mix_coef : 1.0f;
                norm_parts<SPT, E>(x, col, gp, p.norm_dim > 0 ? p.norm_dim : p.cols, p.norm_groups > 1 ? p.norm_groups : 1, p.eps,
                                   gred, 2 + g, T, t);
                const bool store = blockIdx.x == 0 && g == 0;
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; e += 4) {
                        if (store && on[s] && p.d_post_copy)
                            *reinterpret_cast<float4 *>(p.d_post_copy + col[s] + e) = make_float4(x[s][e], x[s][e + 1], x[s][e + 2], x[s][e + 3]);
                        if (p.d_mix_in) {
#pragma unroll
                            for (int k = 0; k < 4; ++k) x[s][e + k] = fmaf(coef, x[s][e + k], mix[s][e + k]);
                        }
                        if (store && on[s] && p.d_resid_out)
                            *reinterpret_cast<float4 *>(p.d_resid_out + col[s] + e) = make_float4(x[s][e], x[s][e + 1], x[s][e + 2], x[s][e + 3]);
                    }
            }
        }
    } else {
        if (p.in_mode == B200_IN_EMBED) {
            long long tok = p.d_tokens[*p.d_pos];
            if (tok < 0 || tok >= p.emb_rows) tok = 0;      // never index outside the table
            const float *er = p.d_emb + tok * (long long)p.cols;
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4) {
                    float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(er + col[s] + e) : make_float4(0, 0, 0, 0);
                    x[s][e] = v4.x * p.emb_scale; x[s][e + 1] = v4.y * p.emb_scale;
                    x[s][e + 2] = v4.z * p.emb_scale; x[s][e + 3] = v4.w * p.emb_scale;
                }
            if constexpr (STR) {
                if (p.d_emb_pos) {
                    float row[SPT][E];
                    load_slices<SPT, E>(row, p.d_emb_pos + (long long)min(*p.d_pos, p.emb_pos_rows - 1) * p.cols, col, on);
#pragma unroll
                    for (int s = 0; s < SPT; ++s)
#pragma unroll
                        for (int e = 0; e < E; ++e) x[s][e] += row[s][e];
                }
                if (p.d_slot_norm_beta) {
                    float w[SPT][E], b[SPT][E];
                    load_slices<SPT, E>(w, p.d_slot_norm_gamma, col, on);
                    load_slices<SPT, E>(b, p.d_slot_norm_beta, col, on);
                    layer_norm<SPT, E>(x, col, w, b, p.norm_dim > 0 ? p.norm_dim : p.cols, p.eps, gred, 2 + g, T, t);
                }
            }
        } else {
            float sacc[SPT][E];
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) sacc[s][e] = 0.0f;
            for (int k = 0; k < p.n_slots; ++k) {
                const float *sl = p.d_slots + (long long)k * p.slot_stride;
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; e += 4) {
                        if (on[s]) {
                            // slots may be written by other GPUs: read them from L2, the point of coherence, never from L1
                            float4 v4 = __ldcg(reinterpret_cast<const float4 *>(sl + col[s] + e));
                            sacc[s][e] += v4.x; sacc[s][e + 1] += v4.y; sacc[s][e + 2] += v4.z; sacc[s][e + 3] += v4.w;
                        }
                    }
            }
            if (p.d_slot_norm_gamma) {
                float ss = 0.0f;
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; ++e) ss = fmaf(sacc[s][e], sacc[s][e], ss);
                ss = group_sum(ss, gred, 2 + g, T, t);
                const float inv = 1.0f / sqrtf(ss / (float)p.cols + p.eps);
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; ++e)
                        if (on[s]) sacc[s][e] = p.d_slot_norm_gamma[col[s] + e] * sacc[s][e] * inv;
            }
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4) {
                    float4 v4 = on[s] ? *reinterpret_cast<const float4 *>(p.d_resid_in + col[s] + e) : make_float4(0, 0, 0, 0);
                    x[s][e] = v4.x + sacc[s][e]; x[s][e + 1] = v4.y + sacc[s][e + 1];
                    x[s][e + 2] = v4.z + sacc[s][e + 2]; x[s][e + 3] = v4.w + sacc[s][e + 3];
                }
        }
        if (blockIdx.x == 0 && g == 0 && p.d_resid_out) {
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4)
                    if (on[s])
                        *reinterpret_cast<float4 *>(p.d_resid_out + col[s] + e) =
                            make_float4(x[s][e], x[s][e + 1], x[s][e + 2], x[s][e + 3]);
        }
        if constexpr (STR) {
            if (p.in_mode == B200_IN_EMBED && p.d_mix_coef) {    // what the first reader takes of the streams, all equal here
                const float c = *p.d_mix_coef;
#pragma unroll
                for (int s = 0; s < SPT; ++s)
#pragma unroll
                    for (int e = 0; e < E; ++e) x[s][e] *= c;
            }
        }
    }
    if ((EXT || STR) && p.d_norm_gamma) {
        if constexpr (STR) layer_norm<SPT, E>(x, col, gm, gb, p.norm_dim > 0 ? p.norm_dim : p.cols, p.eps, gred, 2 + g, T, t);
        if constexpr (EXT)
            norm_parts<SPT, E>(x, col, gm, p.norm_dim > 0 ? p.norm_dim : p.cols, p.norm_groups > 1 ? p.norm_groups : 1, p.eps, gred, 2 + g, T, t);
    } else if (p.d_norm_gamma) {
        float ss = 0.0f;
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) ss = fmaf(x[s][e], x[s][e], ss);
        ss = group_sum(ss, gred, 2 + g, T, t);
        const float inv = 1.0f / sqrtf(ss / (float)p.cols + p.eps);
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) x[s][e] = gm[s][e] * x[s][e] * inv;
    }
    }
    if (p.d_in_copy && blockIdx.x == 0 && g == 0) {
#pragma unroll
        for (int s = 0; s < SPT; ++s)
#pragma unroll
            for (int e = 0; e < E; e += 4)
                if (on[s])
                    *reinterpret_cast<float4 *>(p.d_in_copy + col[s] + e) = make_float4(x[s][e], x[s][e + 1], x[s][e + 2], x[s][e + 3]);
    }
    if (geo.share_x) {
        if (g == 0) {
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4)
                    *reinterpret_cast<float4 *>(xs + (size_t)(s * T + t) * E + e) = make_float4(x[s][e], x[s][e + 1], x[s][e + 2], x[s][e + 3]);
        }
        named_barrier(1, nC);
        if (g != 0) {
#pragma unroll
            for (int s = 0; s < SPT; ++s)
#pragma unroll
                for (int e = 0; e < E; e += 4) {
                    const float4 v4 = *reinterpret_cast<const float4 *>(xs + (size_t)(s * T + t) * E + e);
                    x[s][e] = v4.x; x[s][e + 1] = v4.y; x[s][e + 2] = v4.z; x[s][e + 3] = v4.w;
                }
        }
    }

    // ---------------- consume the ring: group g takes stages g, g+NG, ... ----------------
    float best_v = -INFINITY;
    int best_i = 0x7fffffff;
    // Byte offsets of this thread's slices inside a row. Threads past the end of the row read slice 0
    // (valid memory) against a zero input slice and drop the result.
    uint32_t qoff[SPT], soff[SPT];
#pragma unroll
    for (int s = 0; s < SPT; ++s) {
        const int c = on[s] ? col[s] : 0;
        qoff[s] = (uint32_t)(WT == B200_WT_Q8 ? c : WT == B200_WT_F32 ? 4 * c : 2 * c);
        soff[s] = (uint32_t)p.cols + (uint32_t)(c >> 5) * 2u;   // Q8: scales follow the quants of a row
    }
    const uint32_t ring_s = smem_u32(ring), stride = (uint32_t)p.row_stride;
    for (int i = g, it = 0; i < nst; i += NG, ++it) {
        const int slot = i % nstage;
        const int row0 = r0 + i * RB;
        const int nr = min(RB, r1 - row0);
        float o_resid = 0.0f, o_gate = 0.0f;            // what the gated output adds to and scales by
        if constexpr (EXT) {
            if (p.out_mode == B200_OUT_GATED && wg == 0 && lane < nr) {
                o_resid = p.d_out_resid[row0 + lane];
                o_gate = p.d_out_gate[row0 + lane] + p.d_out_gate_bias[row0 + lane];
            }
        }
        // Streams: lane = row + RB * j holds streams j, j + 32/RB, ... of its row.
        constexpr int LPR = 32 / RB, XS = (B200_MAX_STREAMS + LPR - 1) / LPR;
        float old[STR ? XS : 1];
        if constexpr (STR) {
            if (p.out_mode == B200_OUT_STREAMS && wg == 0) {
#pragma unroll
                for (int k = 0; k < XS; ++k) {
                    const int s = lane / RB + k * LPR, r = lane % RB;
                    old[k] = s < p.n_streams && r < nr ? p.d_streams_in[s * p.streams_in_stride + row0 + r] : 0.0f;
                }
            }
        }
        if (!mbar_wait(&full[slot], (i / nstage) & 1) && p.d_err) *p.d_err = 3;
        const uint32_t sb = ring_s + (uint32_t)slot * geo.slot_bytes;
        // Rows past nr hold stale bytes; they are computed like the others (no predicates in the
        // hot loop), stay in their own reduction lane and are never emitted.
        uint4 wq[RB][SPT];
        uint32_t ws[RB][SPT];
#pragma unroll
        for (int j = 0; j < RB; ++j)
#pragma unroll
            for (int s = 0; s < SPT; ++s) {
                wq[j][s] = lds_128(sb + (uint32_t)j * stride + qoff[s]);
                if (WT == B200_WT_Q8) ws[j][s] = lds_u16(sb + (uint32_t)j * stride + soff[s]);
            }
        float v[RB];
#pragma unroll
        for (int j = 0; j < RB; ++j) {
            float acc = 0.0f;
#pragma unroll
            for (int s = 0; s < SPT; ++s) {
                float d;
                if (WT == B200_WT_Q8) d = __half2float(__ushort_as_half((unsigned short)ws[j][s])) * dot16_q8(wq[j][s], x[s]);
                else if (WT == B200_WT_BF16) d = dot8_bf16(wq[j][s], x[s]);
                else if (WT == B200_WT_F32) d = dot4_f32(wq[j][s], x[s]);
                else d = dot8_f16(wq[j][s], x[s]);
                acc += d;                      // threads past the end of the row hold a zero input slice
            }
            v[j] = acc;
        }
        mbar_arrive(&empty[slot]);             // this thread no longer reads the slot

        const float tot = reduce_rows<RB>(v, lane);
        float *wp = wpart + (size_t)((g * 2 + (it & 1)) * nwg) * RB;
        if (lane < RB) wp[wg * RB + lane] = tot;
        named_barrier(2 + g, T);
        if (wg == 0) {
            float y = 0.0f;
            if (lane < RB)
                for (int w = 0; w < nwg; ++w) y += wp[w * RB + lane];
            const int row = row0 + lane;
            if (p.out_mode == B200_OUT_GLU) {
                const float u = __shfl_down_sync(0xffffffffu, y, 1);
                if (EXT && p.glu_rows > 0 && row >= p.glu_rows) {
                    if (lane < nr) p.d_out2[row - p.glu_rows] = y;
                } else if (lane < nr && !(lane & 1)) {
                    const float a = p.act == 0 ? act_silu(y) : act_gelu_tanh(y);
                    p.d_out[0][p.out_offset + (row >> 1)] = a * u;
                }
            } else if (EXT && p.out_mode == B200_OUT_GATED) {
                if (lane < nr) p.d_out[0][p.out_offset + row] = fmaf(p.resid_alpha, o_resid, sigmoid_f32(o_gate) * y);
            } else if (STR && p.out_mode == B200_OUT_STREAMS) {
                if constexpr (STR) {
                    const int n = p.n_streams, r = lane % RB;
                    const float yr = __shfl_sync(0xffffffffu, y, r);
                    float next = 0.0f;
                    for (int to = 0; to < n; ++to) {
                        float a = 0.0f;
#pragma unroll
                        for (int k = 0; k < XS; ++k) {
                            const int s = lane / RB + k * LPR;
                            if (s < n) a = fmaf(s_conn[s * n + to], old[k], a);
                        }
#pragma unroll
                        for (int o = RB; o < 32; o <<= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
                        a = fmaf(s_conn[n * n + to], yr, a);
                        if (r < nr && lane / RB == to % LPR) p.d_streams_out[to * p.streams_out_stride + row0 + r] = a;
                        next = fmaf(s_conn[n * n + n + to], a, next);
                    }
                    if (lane < nr) p.d_out[0][p.out_offset + row] = next;
                }
            } else if (lane < nr) {
                if (EXT && p.softcap > 0.0f) y = p.softcap * tanhf(y / p.softcap);
                if (STR && p.act == B200_ACT_RELU2) y = act_relu2(y);
                for (int q = 0; q < p.n_out; ++q) p.d_out[q][p.out_offset + row] = y;
                if (better(y, row, best_v, best_i)) { best_v = y; best_i = row; }
            }
        }
    }

    if (!p.d_ticket) return;

    // ---------------- last-block bookkeeping ----------------
    if (p.d_argmax_scratch && wg == 0 && lane < RB) { am_v[g * RB + lane] = best_v; am_i[g * RB + lane] = best_i; }
    // The barrier orders every thread's stores (peers' slots included) before thread 0; its system-wide
    // fence is cumulative, so one fence per block publishes them all before the ticket is taken.
    named_barrier(1, nC);
    if (tid == 0) {
        __threadfence_system();
        if (p.d_argmax_scratch) {
            float bv = am_v[0]; int bi = am_i[0];
            for (int k = 1; k < NG * RB; ++k) if (better(am_v[k], am_i[k], bv, bi)) { bv = am_v[k]; bi = am_i[k]; }
            p.d_argmax_scratch[2 * blockIdx.x] = bv;
            reinterpret_cast<int *>(p.d_argmax_scratch)[2 * blockIdx.x + 1] = bi;
            __threadfence();
        }
        s_last = (atomicAdd(p.d_ticket, 1u) == gridDim.x - 1);
    }
    named_barrier(1, nC);
    if (!s_last || tid >= 32) return;
    __threadfence_system();
    {
        float bv = -INFINITY; int bi = 0x7fffffff;
        if (p.d_argmax_scratch) {
            for (int b = lane; b < (int)gridDim.x; b += 32) {
                const float v = *reinterpret_cast<volatile float *>(p.d_argmax_scratch + 2 * b);
                const int i = *reinterpret_cast<volatile int *>(p.d_argmax_scratch + 2 * b + 1);
                if (better(v, i, bv, bi)) { bv = v; bi = i; }
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) {
                const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
                const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                if (better(ov, oi, bv, bi)) { bv = ov; bi = oi; }
            }
            if (bi == 0x7fffffff) bi = 0;         // nothing compared greater (all NaN): index 0, as the reference's loop
            bi += (int)p.out_offset;              // global row index of a sharded matrix
            if (lane < p.n_argmax_out) { p.d_argmax_val[lane][0] = bv; p.d_argmax_idx[lane][0] = bi; }
        }
        __syncwarp();
        if (lane == 0) {
            const int pos = p.d_pos_rw ? *p.d_pos_rw : 0;
            if (p.d_next_token && pos + 1 >= *p.d_prompt_len) p.d_next_token[pos + 1] = bi;
            if (p.advance_pos) *p.d_pos_rw = pos + 1;
            const unsigned ep = p.d_epoch ? *p.d_epoch : 0u;
            if (p.advance_epoch) *p.d_epoch_rw = ep + 1u;
            *p.d_ticket = 0u;
            if (p.n_signal > 0) {
                __threadfence_system();
                const unsigned want = ep * (unsigned)p.epoch_mul + (unsigned)p.epoch_add;
                for (int q = 0; q < p.n_signal; ++q) st_release_sys(p.d_signal_flags[q] + p.signal_index, want);
            }
        }
    }
}

template <int WT, int SPT, int RB, int MAXT, int FAM>
int launch(const b200_matvec_args &a, const Geometry &geo, int grid, cudaStream_t st)
{
    const int nwg = geo.T / 32;
    const size_t smem = (size_t)geo.nstage * geo.slot_bytes + (size_t)geo.nstage * 16 +
                        ((size_t)geo.NG * 2 * nwg * RB + (size_t)geo.NG * 32 + (size_t)geo.NG * RB * 2) * sizeof(float) +
                        (geo.share_x ? (size_t)SPT * geo.T * (WT == B200_WT_Q8 ? 16 : WT == B200_WT_F32 ? 4 : 8) * sizeof(float) : 0);
    auto kern = matvec_kernel<WT, SPT, RB, MAXT, FAM>;
    if (smem > 220 * 1024) return B200_E_TOOLARGE;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(grid);
    cfg.blockDim = dim3(geo.NG * geo.T + 32);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.use_pdl ? 1 : 0;
    ++g_b200_launches;
    return (int)cudaLaunchKernelEx(&cfg, kern, a, geo);
}

template <int WT, int SPT, int RB, int FAM>
int launch_by_size(const b200_matvec_args &a, const Geometry &geo, int grid, cudaStream_t st)
{
    const int threads = geo.NG * geo.T + 32;
    if (threads <= 672) return launch<WT, SPT, RB, 672, FAM>(a, geo, grid, st);
    return launch<WT, SPT, RB, 1024, FAM>(a, geo, grid, st);
}

template <int WT, int SPT, int FAM = FAM_PLAIN>
int launch_by_rows(const b200_matvec_args &a, const Geometry &geo, int rb, int grid, cudaStream_t st)
{
    switch (rb) {
    case 8: return launch_by_size<WT, SPT, 8, FAM>(a, geo, grid, st);
    case 4: return launch_by_size<WT, SPT, 4, FAM>(a, geo, grid, st);
    case 2: return launch_by_size<WT, SPT, 2, FAM>(a, geo, grid, st);
    default: return launch_by_size<WT, SPT, 1, FAM>(a, geo, grid, st);
    }
}


// BF16 / F32 weights
template <int FAM>
int launch_typed(const b200_matvec_args &a, const Geometry &geo, int spt, int rb, int grid, cudaStream_t st)
{
    if (a.wtype == B200_WT_BF16)
        return spt == 1 ? launch_by_rows<B200_WT_BF16, 1, FAM>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_BF16, 2, FAM>(a, geo, rb, grid, st);
    return spt == 1 ? launch_by_rows<B200_WT_F32, 1, FAM>(a, geo, rb, grid, st)
         : spt == 2 ? launch_by_rows<B200_WT_F32, 2, FAM>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_F32, 4, FAM>(a, geo, rb, grid, st);
}
int launch_ext(const b200_matvec_args &a, const Geometry &geo, int spt, int rb, int grid, cudaStream_t st);        // matvec_ext.cu
int launch_streams(const b200_matvec_args &a, const Geometry &geo, int spt, int rb, int grid, cudaStream_t st);    // matvec_streams.cu

} // namespace b200_mv
