// Grouped-query attention with normed queries and keys (sm_100a): heads of any size, a per-position query factor, an
// optional cap on the scores, key and value rows cached in bfloat16 or fp32.
//
// Decode, one launch: a cluster of blocks serves the query heads of one key/value head (up to HB of them) over its share
// of the cached positions; the first rows are fetched before the kernel waits for its predecessor. The newest position's
// key and value come from the projection; the block that owns it stores them. Two forms of the inner part:
//   gqa_decode_mma   bfloat16, heads up to 256 wide: sixteen query heads are the rows of the tensor-core tiles, every warp
//                    takes tiles of sixteen positions of its own
//   gqa_decode       fp32, and wider heads: a key row lies across a group of LPK lanes, sixteen bytes each; the scores of a
//                    batch (HB heads x U positions) are summed over the group by folding, so that every lane ends up with
//                    scores of its own to cap and exponentiate
// Warps or groups merge through shared memory, blocks through the cluster's distributed shared memory, and clusters
// (long sequences only) through partial records and a ticket: the last block to finish merges.
//
// Prompt portions: gqa_prep writes cache rows and query rows of all tokens, the attention is that of row_attention.cuh.
#include "row_attention.cuh"

#include <cooperative_groups.h>

namespace cg = cooperative_groups;

namespace {

constexpr int BLOCK_KEYS = 512;    // positions per block before a second cluster is worth its merge
constexpr int MAX_SPLITS = 64;
constexpr int MAX_CLUSTER = 8;
constexpr int MAX_HEADS = 16;      // query heads of a block
constexpr int THREADS = 256, WARPS = THREADS / 32;
constexpr int DEPTH = 4;           // batches of positions in flight

__host__ __device__ __forceinline__ int part_stride(int vdim) { return up8(vdim) + 8; }

// Elements col .. col + E of a projection's vector of n; zeros past its end.
template <int E>
__device__ __forceinline__ void load_part(float (&x)[E], const float *v, int col, int n)
{
#pragma unroll
    for (int e = 0; e < E; ++e) x[e] = col + e < n ? v[col + e] : 0.0f;
}

template <typename T> __device__ __forceinline__ float rounded(float x) { return (float)(T)x; }

// The two transcendental functions of a score: the bfloat16 form through the fast exponential, fp32 with the library's.
template <int WT> __device__ __forceinline__ float weight_of(float x) { return WT == B200_WT_F32 ? expf(x) : ex2(x * 1.4426950408889634f); }
template <int WT> __device__ __forceinline__ float capped(float s, float cap)
{
    if (cap <= 0.0f) return s;
    return WT == B200_WT_F32 ? cap * tanhf(s / cap) : soft_cap(s, 2.0f * 1.4426950408889634f / cap, cap);
}

// Which positions of 0 .. n - 1 this block takes: a cluster's contiguous share, a block's contiguous part of it.
struct Share { int split, rank, active, lo, hi; };           // active: clusters that have any
__device__ __forceinline__ Share share_of(const b200_gqa_args &p, int n, int cluster_size)
{
    Share r;
    r.split = blockIdx.x / cluster_size; r.rank = blockIdx.x % cluster_size;
    const int per = max((n + p.n_split - 1) / p.n_split, cluster_size * BLOCK_KEYS);
    r.active = (n + per - 1) / per;
    const int lo = min(r.split * per, n), hi = min(lo + per, n), each = (hi - lo + cluster_size - 1) / cluster_size;
    r.lo = min(lo + r.rank * each, hi); r.hi = min(r.lo + each, hi);
    return r;
}

// The end of a block's work: rec [ng][stride][v8] holds sums of ng parts, sm / st [heads][ng] their maxima and totals
// (shared memory, written before a __syncthreads). sw [nh][ng] is shared scratch, inbox [cluster][inbox_of(..)] what
// the cluster's blocks send to this one (nh v8 + MAX_CLUSTER floats hold it): each block merges a share of the columns. All THREADS come here, and have
// passed cluster_here() before.
struct Merge { const float *rec, *sm, *st; float *sw, *inbox; int ng, stride, nh, h0; };
__host__ __device__ __forceinline__ int inbox_of(int nh, int vdim, int cluster_size) { return (nh * up8(vdim) + cluster_size - 1) / cluster_size; }
__device__ __forceinline__ void cluster_here() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
template <int WT>
__device__ __forceinline__ void merge_all(const b200_gqa_args &p, const Merge &g, const Share &r, int cluster_size)
{
    __shared__ float im[MAX_CLUSTER][MAX_HEADS], it[MAX_CLUSTER][MAX_HEADS];
    __shared__ int s_last;
    cg::cluster_group cluster = cg::this_cluster();
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");      // every block of the cluster has started
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, v8 = up8(p.vdim);
    for (int i = warp; i < g.nh; i += WARPS) {
        float mt = -INFINITY, t = 0.0f;
        for (int k = lane; k < g.ng; k += 32) mt = fmaxf(mt, g.sm[i * g.ng + k]);
        mt = warp_max(mt);
        for (int k = lane; k < g.ng; k += 32) {
            const float m = g.sm[i * g.ng + k], f = m == -INFINITY ? 0.0f : weight_of<WT>(m - mt);
            g.sw[i * g.ng + k] = f;
            t = fmaf(f, g.st[i * g.ng + k], t);
        }
        t = warp_sum(t);
        if (lane < cluster_size) { *cluster.map_shared_rank(&im[r.rank][i], lane) = mt; *cluster.map_shared_rank(&it[r.rank][i], lane) = t; }
    }
    __syncthreads();
    const int PS = part_stride(p.vdim), n = g.nh * v8, box = inbox_of(g.nh, p.vdim, cluster_size);
    for (int e = tid; e < n; e += THREADS) {
        const int i = e / v8, col = e % v8;
        float a = 0.0f;
#pragma unroll 8
        for (int k = 0; k < g.ng; ++k) a = fmaf(g.sw[i * g.ng + k], g.rec[(size_t)(k * g.stride + i) * v8 + col], a);
        *cluster.map_shared_rank(g.inbox + r.rank * box + e % box, e / box) = a;
    }
    cluster.sync();
    for (int e = r.rank * box + tid; e < min((r.rank + 1) * box, n); e += THREADS) {
        const int i = e / v8, col = e % v8;
        float mt = -INFINITY, a = 0.0f, t = 0.0f;
#pragma unroll
        for (int c = 0; c < MAX_CLUSTER; ++c) mt = fmaxf(mt, c < cluster_size ? im[c][i] : -INFINITY);
#pragma unroll
        for (int c = 0; c < MAX_CLUSTER; ++c)
            if (c < cluster_size) {
                const float f = im[c][i] == -INFINITY ? 0.0f : weight_of<WT>(im[c][i] - mt);
                a = fmaf(f, g.inbox[c * box + e % box], a);
                t = fmaf(f, it[c][i], t);
            }
        if (r.active == 1) {
            if (col < p.vdim) p.d_out[(size_t)(g.h0 + i) * p.vdim + col] = a / t;
        } else {
            float *part = p.d_part + ((size_t)(g.h0 + i) * p.n_split + r.split) * PS;
            part[col] = a;
            if (col == 0) { part[v8] = mt; part[v8 + 1] = t; }
        }
    }
    if (r.active == 1) return;
    // the clusters
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(p.d_tickets + blockIdx.y, 1u) == (unsigned)(r.active * cluster_size) - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) p.d_tickets[blockIdx.y] = 0u;
    for (int e = tid; e < g.nh * p.vdim; e += THREADS) {
        const int i = e / p.vdim, col = e % p.vdim;
        const float *part = p.d_part + (size_t)(g.h0 + i) * p.n_split * PS;
        float mt = -INFINITY, a = 0.0f, t = 0.0f;
#pragma unroll 8
        for (int s = 0; s < r.active; ++s) mt = fmaxf(mt, __ldcg(part + (size_t)s * PS + v8));
#pragma unroll 8
        for (int s = 0; s < r.active; ++s) {
            const float f = weight_of<WT>(__ldcg(part + (size_t)s * PS + v8) - mt);
            a = fmaf(f, __ldcg(part + (size_t)s * PS + col), a);
            t = fmaf(f, __ldcg(part + (size_t)s * PS + v8 + 1), t);
        }
        p.d_out[(size_t)(g.h0 + i) * p.vdim + col] = a / t;
    }
}

// v[n] holds this lane's part of value n. Sums them over the LPK lanes of a group; lane sl ends up with the values
// (sl / REP) * VL + r in v[r], r < VL, where VL = max(NV / LPK, 1) and REP = max(LPK / NV, 1) lanes hold the same ones.
template <int NV, int LPK>
__device__ __forceinline__ void fold(float (&v)[NV], int lane)
{
    int n = NV;
#pragma unroll
    for (int o = LPK / 2; o >= 1; o >>= 1) {
        if (n > 1) {
            n /= 2;
            const bool up = (lane & o) != 0;
#pragma unroll
            for (int k = 0; k < n; ++k) {
                const float send = up ? v[k] : v[k + n], keep = up ? v[k + n] : v[k];
                v[k] = keep + __shfl_xor_sync(0xffffffffu, send, o);
            }
        } else v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
}

// HB heads a block, NS slices of sixteen bytes per lane and row, LPK lanes per row.
template <int WT, int HB, int NS, int LPK>
__global__ void __launch_bounds__(THREADS) gqa_decode_kernel(const __grid_constant__ b200_gqa_args p, int cluster_size, int chunks)
{
    using El = Elem<WT>;
    using T = typename El::T;
    constexpr int E = El::E, U = 4 / NS;                     // U positions of a group at a time
    constexpr int NV = HB * U, VL = NV > LPK ? NV / LPK : 1, REP = LPK > NV ? LPK / NV : 1;
    constexpr int LH = LPK / HB;                             // lanes that hold one head's scores
    constexpr int GPW = 32 / LPK, NG = WARPS * GPW;          // groups of a warp, of the block
    static_assert(VL <= U && LH >= 1, "a lane's values belong to one head");
    // [NG][HB][up8(vdim)] sums; [HB][NG] weights; inbox; [DEPTH][U][NS][key, value][THREADS] rows in flight
    extern __shared__ __align__(16) float sh[];
    __shared__ float sm[HB][NG], st[HB][NG];
    pdl_launch_dependents();
    const int pos = *p.d_pos;
    if (pos < 0 || pos >= p.max_seq) return;
    const Share share = share_of(p, pos + 1, cluster_size);
    if (share.split >= share.active) return;                 // the whole cluster
    cluster_here();
    const int k_lo = share.lo, k_hi = min(share.hi, pos);    // cached ones
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kg = warp * GPW + lane / LPK, sl = lane % LPK, gbase = lane - sl;
    const int kvh = blockIdx.y / chunks, h_in0 = (blockIdx.y % chunks) * HB, group = p.heads / p.kv_heads;
    const int h0 = kvh * group + h_in0, nh = min(HB, group - h_in0);
    const int d8 = up8(p.dim), v8 = up8(p.vdim);
    const T *kc = static_cast<const T *>(p.d_k_cache) + (size_t)kvh * p.max_seq * d8;
    const T *vc = static_cast<const T *>(p.d_v_cache) + (size_t)kvh * p.max_seq * v8;

    float *sw = sh + (size_t)NG * HB * v8, *inbox = sw + HB * NG;
    uint4 *ring = reinterpret_cast<uint4 *>(inbox + HB * v8 + MAX_CLUSTER) + tid;
    auto slot = [&](int b, int u, int s, int kv) { return ring + ((((b % DEPTH) * U + u) * NS + s) * 2 + kv) * THREADS; };
    auto fetch = [&](int b) {                                // batch b: positions k_lo + b U NG + kg, + NG, ...; zeros past the end
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int j = k_lo + (b * U + u) * NG + kg;
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                const int col = (sl + s * LPK) * E;
                const bool k_on = j < k_hi && col < d8, v_on = j < k_hi && col < v8;
                cp16(smem_u32(slot(b, u, s, 0)), k_on ? kc + (size_t)j * d8 + col : kc, k_on);
                cp16(smem_u32(slot(b, u, s, 1)), v_on ? vc + (size_t)j * v8 + col : vc, v_on);
            }
        }
    };
#pragma unroll
    for (int b = 0; b < DEPTH; ++b) {
        if (k_lo + b * U * NG < k_hi) fetch(b);
        cp_commit();
    }
    float gq[NS][E], gk[NS][E];
#pragma unroll
    for (int s = 0; s < NS; ++s) { load_part<E>(gq[s], p.d_q_gamma, (sl + s * LPK) * E, p.dim); load_part<E>(gk[s], p.d_k_gamma, (sl + s * LPK) * E, p.dim); }
    const float factor = p.scale * (p.d_q_scale ? p.d_q_scale[pos] : 1.0f);
    pdl_wait();

    // queries, normed: sums of squares of all heads folded together
    float q[HB][NS][E];
    {
        float ss[HB];
#pragma unroll
        for (int i = 0; i < HB; ++i) {
            ss[i] = 0.0f;
#pragma unroll
            for (int s = 0; s < NS; ++s) load_part<E>(q[i][s], p.d_q + (size_t)(h0 + min(i, nh - 1)) * p.dim, (sl + s * LPK) * E, p.dim);
        }
#pragma unroll
        for (int i = 0; i < HB; ++i)
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) ss[i] = fmaf(q[i][s][e], q[i][s][e], ss[i]);
        fold<HB, LPK>(ss, lane);                             // lane holds head sl / LH
        const float mine = factor / sqrtf(ss[0] / (float)p.dim + p.eps);
#pragma unroll
        for (int i = 0; i < HB; ++i) {
            const float inv = __shfl_sync(0xffffffffu, mine, gbase + i * LH);
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) q[i][s][e] = gq[s][e] * (q[i][s][e] * inv);
        }
    }

    float m = -INFINITY, l = 0.0f;                           // of this lane's head; l: this lane's share
    float2 acc[HB][NS][E / 2];
#pragma unroll
    for (int i = 0; i < HB; ++i)
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E / 2; ++e) acc[i][s][e] = make_float2(0.0f, 0.0f);
    // U positions: key(u, s, x) and value(u, s, x) give a slice as fp32, valid(u) tells whether the group has that position
    auto batch = [&](auto key, auto value, auto valid) {
        float s_v[NV];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float2 a[HB];
#pragma unroll
            for (int i = 0; i < HB; ++i) a[i] = make_float2(0.0f, 0.0f);
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                float x[E];
                key(u, s, x);
#pragma unroll
                for (int i = 0; i < HB; ++i)
#pragma unroll
                    for (int e = 0; e < E; e += 2) a[i] = __ffma2_rn(make_float2(x[e], x[e + 1]), make_float2(q[i][s][e], q[i][s][e + 1]), a[i]);
            }
#pragma unroll
            for (int i = 0; i < HB; ++i) s_v[i * U + u] = a[i].x + a[i].y;
        }
        fold<NV, LPK>(s_v, lane);
        float mt = m;
#pragma unroll
        for (int r = 0; r < VL; ++r) {
            const int u = ((sl / REP) * VL + r) % U;
            s_v[r] = valid(u) ? capped<WT>(s_v[r], p.softcap) : -INFINITY;
            mt = fmaxf(mt, s_v[r]);
        }
#pragma unroll
        for (int o = LH / 2; o >= 1; o >>= 1) mt = fmaxf(mt, __shfl_xor_sync(0xffffffffu, mt, o));
        const float base = mt == -INFINITY ? 0.0f : mt, corr = weight_of<WT>(m - base);
        m = mt;
        l *= corr;
#pragma unroll
        for (int r = 0; r < VL; ++r) {
            s_v[r] = weight_of<WT>(s_v[r] - base);
            if (sl % REP == 0) l += s_v[r];
        }
#pragma unroll
        for (int i = 0; i < HB; ++i) {
            const float c = __shfl_sync(0xffffffffu, corr, gbase + i * LH);
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E / 2; ++e) { acc[i][s][e].x *= c; acc[i][s][e].y *= c; }
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            float w[HB];
#pragma unroll
            for (int i = 0; i < HB; ++i) w[i] = __shfl_sync(0xffffffffu, s_v[(i * U + u) % VL], gbase + (i * U + u) / VL * REP);
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                float x[E];
                value(u, s, x);
#pragma unroll
                for (int i = 0; i < HB; ++i)
#pragma unroll
                    for (int e = 0; e < E / 2; ++e) acc[i][s][e] = __ffma2_rn(make_float2(w[i], w[i]), make_float2(x[2 * e], x[2 * e + 1]), acc[i][s][e]);
            }
        }
    };
    // every group of a warp takes the same number of trips: the shuffles are warp-wide
    for (int b = 0; k_lo + b * U * NG < k_hi; ++b) {
        cp_wait<DEPTH - 1>();
        batch([&](int u, int s, float (&x)[E]) { El::unpack(*slot(b, u, s, 0), x); }, [&](int u, int s, float (&x)[E]) { El::unpack(*slot(b, u, s, 1), x); },
              [&](int u) { return k_lo + (b * U + u) * NG + kg < k_hi; });
        if (k_lo + (b + DEPTH) * U * NG < k_hi) fetch(b + DEPTH);
        cp_commit();
    }
    if (share.lo <= pos && pos < share.hi && warp == 0) {    // the newest position, by the first group
        float kx[NS][E], vx[NS][E], ss = 0.0f;
#pragma unroll
        for (int s = 0; s < NS; ++s) {
            load_part<E>(kx[s], p.d_k + (size_t)kvh * p.dim, (sl + s * LPK) * E, p.dim);
            load_part<E>(vx[s], p.d_v + (size_t)kvh * p.vdim, (sl + s * LPK) * E, p.vdim);
#pragma unroll
            for (int e = 0; e < E; ++e) ss = fmaf(kx[s][e], kx[s][e], ss);
        }
#pragma unroll
        for (int o = 1; o < LPK; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.0f / sqrtf(ss / (float)p.dim + p.eps);
        const bool store = lane < LPK && h_in0 == 0;
        T *kd = static_cast<T *>(p.d_k_cache) + ((size_t)kvh * p.max_seq + pos) * d8, *vd = static_cast<T *>(p.d_v_cache) + ((size_t)kvh * p.max_seq + pos) * v8;
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) {                    // padding columns are zeros
                const int col = (sl + s * LPK) * E + e;
                kx[s][e] = rounded<T>(gk[s][e] * (kx[s][e] * inv));
                vx[s][e] = rounded<T>(vx[s][e]);
                if (store && col < d8) kd[col] = (T)kx[s][e];
                if (store && col < v8) vd[col] = (T)vx[s][e];
            }
        batch([&](int, int s, float (&x)[E]) {
#pragma unroll
                  for (int e = 0; e < E; ++e) x[e] = kx[s][e];
              },
              [&](int, int s, float (&x)[E]) {
#pragma unroll
                  for (int e = 0; e < E; ++e) x[e] = vx[s][e];
              },
              [&](int u) { return u == 0 && lane < LPK; });
    }

    // the groups of the block
#pragma unroll
    for (int o = LH / 2; o >= 1; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
    if (sl % LH == 0) { sm[sl / LH][kg] = m; st[sl / LH][kg] = l; }
#pragma unroll
    for (int i = 0; i < HB; ++i)
#pragma unroll
        for (int s = 0; s < NS; ++s) {
            const int col = (sl + s * LPK) * E;
            if (col < v8) {
                float *rec = sh + (size_t)(kg * HB + i) * v8 + col;
#pragma unroll
                for (int e = 0; e < E; e += 4)
                    *reinterpret_cast<float4 *>(rec + e) = make_float4(acc[i][s][e / 2].x, acc[i][s][e / 2].y, acc[i][s][e / 2 + 1].x, acc[i][s][e / 2 + 1].y);
            }
        }
    __syncthreads();
    merge_all<WT>(p, Merge{sh, &sm[0][0], &st[0][0], sw, inbox, NG, HB, nh, h0}, share, cluster_size);
}

// bfloat16 on the tensor cores. Shared: query rows [16][dqs]; the newest key and value; then per warp `stages` tiles of
// sixteen key rows [16][dqs] and value rows [16][DV + 8] (rows 16 bytes off a multiple of 32: ldmatrix is conflict-free).
// The tiles' memory holds the warps' results afterwards.
constexpr int TK = 16;
template <int DV>
__global__ void __launch_bounds__(THREADS) gqa_decode_mma_kernel(const __grid_constant__ b200_gqa_args p, int cluster_size, int chunks, int dqs, int stages)
{
    using T = __nv_bfloat16;
    constexpr int VS = DV + 8;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float sm[MAX_HEADS][WARPS], st[MAX_HEADS][WARPS], sw[MAX_HEADS][WARPS];
    pdl_launch_dependents();
    const int pos = *p.d_pos;
    if (pos < 0 || pos >= p.max_seq) return;
    const Share share = share_of(p, pos + 1, cluster_size);
    if (share.split >= share.active) return;                 // the whole cluster
    cluster_here();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int group = p.heads / p.kv_heads, kvh = blockIdx.y / chunks, h_in0 = (blockIdx.y % chunks) * MAX_HEADS;
    const int h0 = kvh * group + h_in0, nh = min(MAX_HEADS, group - h_in0);
    const int d8 = up8(p.dim), v8 = up8(p.vdim), dqk = dqs - 8;
    T *qs = reinterpret_cast<T *>(smem), *newest = qs + TK * dqs;            // [dqs] key, [VS] value
    float *inbox = reinterpret_cast<float *>(newest + dqs + VS);
    T *tiles = reinterpret_cast<T *>(inbox + nh * v8 + MAX_CLUSTER);
    const uint32_t mine = smem_u32(tiles) + (uint32_t)(warp * stages * TK * (dqs + VS)) * 2;
    const T *kc = static_cast<const T *>(p.d_k_cache) + (size_t)kvh * p.max_seq * d8;
    const T *vc = static_cast<const T *>(p.d_v_cache) + (size_t)kvh * p.max_seq * v8;
    auto key_slot = [&](int t) { return mine + (uint32_t)((t % stages) * TK * (dqs + VS)) * 2; };
    auto value_slot = [&](int t) { return key_slot(t) + TK * dqs * 2; };
    // tile t of this warp: positions share.lo + (t * WARPS + warp) * TK ..; rows not cached (yet) hold zeros
    const int first = share.lo + warp * TK;
    auto fetch = [&](int t) {
        const int j0 = first + t * WARPS * TK;
        const uint32_t kd = key_slot(t), vd = value_slot(t);
        const int sq = dqk / 8, sv = DV / 8;
        for (int e = lane; e < TK * sq; e += 32) {
            const int r = e / sq, c = e % sq;
            const bool on = j0 + r < share.hi && j0 + r < pos && c * 8 < d8;
            cp16(kd + (r * dqs + c * 8) * 2, on ? kc + (size_t)(j0 + r) * d8 + c * 8 : kc, on);
        }
        for (int e = lane; e < TK * sv; e += 32) {
            const int r = e / sv, c = e % sv;
            const bool on = j0 + r < share.hi && j0 + r < pos && c * 8 < v8;
            cp16(vd + (r * VS + c * 8) * 2, on ? vc + (size_t)(j0 + r) * v8 + c * 8 : vc, on);
        }
    };
    for (int t = 0; t < stages; ++t) {
        if (first + t * WARPS * TK < share.hi) fetch(t);
        cp_commit();
    }
    const float factor = p.d_q_scale ? p.d_q_scale[pos] : 1.0f;
    // the rows of the projection this block prepares, a warp each: its query heads, and the newest key and value where it
    // owns the position
    const bool owner = share.lo <= pos && pos < share.hi;
    const int n_rows = nh + (owner ? 2 : 0);
    constexpr int HELD = DV > 128 ? 8 : 4;                   // elements a lane keeps in registers
    float gamma[HELD];
    auto fetch_gamma = [&](int i) {
        const float *g = i < nh ? p.d_q_gamma : p.d_k_gamma;
#pragma unroll
        for (int k = 0; k < HELD; ++k) gamma[k] = i <= nh && lane + 32 * k < p.dim ? g[lane + 32 * k] : 1.0f;
    };
    fetch_gamma(warp);
    for (int e = tid; e < (TK - nh) * (dqs / 8); e += THREADS) *reinterpret_cast<uint4 *>(qs + nh * dqs + e * 8) = make_uint4(0, 0, 0, 0);
    pdl_wait();

    for (int i = warp; i < n_rows; i += WARPS) {
        const bool key = i == nh, value = i > nh;
        const int n = value ? p.vdim : p.dim, n8 = value ? v8 : d8, width = value ? VS : dqs;
        const float *x = value ? p.d_v + (size_t)kvh * p.vdim : key ? p.d_k + (size_t)kvh * p.dim : p.d_q + (size_t)(h0 + i) * p.dim;
        T *out = value ? newest + dqs : key ? newest : qs + i * dqs;
        T *row = value ? static_cast<T *>(p.d_v_cache) + ((size_t)kvh * p.max_seq + pos) * v8 : static_cast<T *>(p.d_k_cache) + ((size_t)kvh * p.max_seq + pos) * d8;
        float held[HELD], ss = 0.0f;
#pragma unroll
        for (int k = 0; k < HELD; ++k) {
            held[k] = lane + 32 * k < n ? x[lane + 32 * k] : 0.0f;
            ss = fmaf(held[k], held[k], ss);
        }
        for (int e = lane + 32 * HELD; e < n; e += 32) ss = fmaf(x[e], x[e], ss);
        if (i != warp) fetch_gamma(i);
        const float inv = value ? 1.0f : (key ? 1.0f : factor) / sqrtf(warp_sum(ss) / (float)n + p.eps);
        auto put = [&](int e, float v) {
            out[e] = __float2bfloat16_rn(v);
            if (i >= nh && h_in0 == 0 && e < n8) row[e] = __float2bfloat16_rn(v);
        };
#pragma unroll
        for (int k = 0; k < HELD; ++k)
            if (lane + 32 * k < width) put(lane + 32 * k, held[k] * inv * gamma[k]);
        for (int e = lane + 32 * HELD; e < width; e += 32) put(e, e < n ? x[e] * inv * (value ? 1.0f : key ? p.d_k_gamma[e] : p.d_q_gamma[e]) : 0.0f);
    }
    __syncthreads();

    float o[DV / 8][4], mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) o[i][k] = 0.0f;
    const uint32_t qaddr = smem_u32(qs) + ((lane & 15) * dqs + (lane >> 4) * 8) * 2;
    const bool capping = p.softcap > 0.0f;
    const float cap_in = capping ? 2.0f * 1.4426950408889634f * p.scale / p.softcap : 0.0f;
    const float sc = (capping ? 1.0f : p.scale) * 1.4426950408889634f;
    for (int t = 0; first + t * WARPS * TK < share.hi; ++t) {
        if (stages == 2) cp_wait<1>();
        else cp_wait<0>();
        __syncwarp();
        const int j0 = first + t * WARPS * TK;
        if (owner && j0 <= pos && pos < j0 + TK) {           // the newest position is in this tile
            const int r = pos - j0;
            for (int e = lane; e < dqk / 8; e += 32)
                *reinterpret_cast<uint4 *>(tiles + (size_t)(warp * stages + t % stages) * TK * (dqs + VS) + r * dqs + e * 8) = *reinterpret_cast<const uint4 *>(newest + e * 8);
            for (int e = lane; e < DV / 8; e += 32)
                *reinterpret_cast<uint4 *>(tiles + (size_t)(warp * stages + t % stages) * TK * (dqs + VS) + TK * dqs + r * VS + e * 8) =
                    *reinterpret_cast<const uint4 *>(newest + dqs + e * 8);
        }
        __syncwarp();
        float s[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
        const uint32_t kaddr = key_slot(t) + (((lane & 7) + ((lane >> 4) << 3)) * dqs + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll 4
        for (int kk = 0; kk < dqk; kk += 16) {
            uint32_t a[4], b[4];
            ldsm4(qaddr + kk * 2, a);
            ldsm4(kaddr + kk * 2, b);
            mma_bf16(s[0], a, b[0], b[1]);
            mma_bf16(s[1], a, b[2], b[3]);
        }
        const int n = share.hi - j0 - (lane & 3) * 2;        // columns of this lane that exist
        float mt[2] = {mx[0], mx[1]};
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (capping) s[c][k] = soft_cap(s[c][k], cap_in, p.softcap);
                if (c * 8 + (k & 1) >= n) s[c][k] = -INFINITY;
                mt[k >> 1] = fmaxf(mt[k >> 1], s[c][k]);
            }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 1));
            mt[r] = fmaxf(mt[r], __shfl_xor_sync(0xffffffffu, mt[r], 2));
        }
        // a tile holds at least one position: the maxima are finite from here on
        const float corr[2] = {ex2((mx[0] - mt[0]) * sc), ex2((mx[1] - mt[1]) * sc)};
        mx[0] = mt[0]; mx[1] = mt[1];
        l[0] *= corr[0]; l[1] *= corr[1];
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                s[c][k] = ex2((s[c][k] - mt[k >> 1]) * sc);
                l[k >> 1] += s[c][k];
            }
        if (t > 0)
#pragma unroll
            for (int i = 0; i < DV / 8; ++i) { o[i][0] *= corr[0]; o[i][1] *= corr[0]; o[i][2] *= corr[1]; o[i][3] *= corr[1]; }
        const uint32_t a[4] = {pack_bf16(s[0][0], s[0][1]), pack_bf16(s[0][2], s[0][3]), pack_bf16(s[1][0], s[1][1]), pack_bf16(s[1][2], s[1][3])};
        const uint32_t vaddr = value_slot(t) + ((lane & 15) * VS + (lane >> 4) * 8) * 2;
#pragma unroll
        for (int c = 0; c < DV / 16; ++c) {
            uint32_t b[4];
            ldsm4_t(vaddr + c * 32, b);
            mma_bf16(o[2 * c], a, b[0], b[1]);
            mma_bf16(o[2 * c + 1], a, b[2], b[3]);
        }
        __syncwarp();                                        // the slot is overwritten next
        if (first + (t + stages) * WARPS * TK < share.hi) fetch(t + stages);
        cp_commit();
    }
    // maxima as the merge expects them: of scores whose weight is exp(score)
    const float unit = sc / 1.4426950408889634f;
    __syncthreads();                                         // every warp is done with its tiles
    float *rec = reinterpret_cast<float *>(tiles);           // [WARPS][nh][v8]
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
        l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
        const int i = (lane >> 2) + 8 * r;
        if (i >= nh) continue;
        if ((lane & 3) == 0) { sm[i][warp] = mx[r] * unit; st[i][warp] = l[r]; }
#pragma unroll
        for (int c = 0; c < DV / 8; ++c) {
            const int col = c * 8 + (lane & 3) * 2;
            if (col < v8) *reinterpret_cast<float2 *>(rec + (size_t)(warp * nh + i) * v8 + col) = make_float2(o[c][2 * r], o[c][2 * r + 1]);
        }
    }
    __syncthreads();
    merge_all<B200_WT_BF16>(p, Merge{rec, &sm[0][0], &st[0][0], &sw[0][0], inbox, WARPS, nh, nh, h0}, share, cluster_size);
}

// ------------------------------------------------------------------------------------------------ rows

// One block per token, a warp per head: query heads to d_q_rows, key and value heads to the cache.
template <int WT>
__global__ void __launch_bounds__(THREADS) gqa_prep_kernel(const __grid_constant__ b200_gqa_args p)
{
    using T = typename Elem<WT>::T;
    const int m = blockIdx.x, pos = p.pos0 + m, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int d8 = up8(p.dim), v8 = up8(p.vdim);
    const float factor = p.d_q_scale ? p.d_q_scale[pos] : 1.0f;
    for (int i = warp + blockIdx.y * WARPS; i < p.heads + 2 * p.kv_heads; i += WARPS * gridDim.y) {
        const bool query = i < p.heads, value = i >= p.heads + p.kv_heads;
        const int g = query ? i : value ? i - p.heads - p.kv_heads : i - p.heads;
        const int n = value ? p.vdim : p.dim, n8 = value ? v8 : d8;
        const float *x = (query ? p.d_q : value ? p.d_v : p.d_k) + (size_t)m * p.proj_ld + (size_t)g * n;
        T *out = query ? static_cast<T *>(p.d_q_rows) + ((size_t)m * p.heads + g) * d8
                       : static_cast<T *>(value ? p.d_v_cache : p.d_k_cache) + ((size_t)g * p.max_seq + pos) * n8;
        float held[8], ss = 0.0f;                            // 256 elements of a head in registers
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int e = lane + 32 * k;
            held[k] = e < n ? __ldg(x + e) : 0.0f;
            ss = fmaf(held[k], held[k], ss);
        }
        for (int e = lane + 256; e < n; e += 32) ss = fmaf(x[e], x[e], ss);
        if (value) {
#pragma unroll
            for (int k = 0; k < 8; ++k)
                if (lane + 32 * k < n8) out[lane + 32 * k] = (T)held[k];
            for (int e = lane + 256; e < n8; e += 32) out[e] = (T)(e < n ? x[e] : 0.0f);
            continue;
        }
        const float *gamma = query ? p.d_q_gamma : p.d_k_gamma;
        const float inv = (query ? factor : 1.0f) / sqrtf(warp_sum(ss) / (float)n + p.eps);
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            const int e = lane + 32 * k;
            if (e < n8) out[e] = (T)(e < n ? __ldg(gamma + e) * (held[k] * inv) : 0.0f);
        }
        for (int e = lane + 256; e < n8; e += 32) out[e] = (T)(e < n ? gamma[e] * (x[e] * inv) : 0.0f);
    }
}

// ------------------------------------------------------------------------------------------------ host side

bool shape_ok(const b200_gqa_args *a)
{
    return a && (a->wtype == B200_WT_BF16 || a->wtype == B200_WT_F32) && a->heads > 0 && a->kv_heads > 0 && a->heads % a->kv_heads == 0 &&
           a->dim > 0 && a->vdim > 0 && a->max_seq > 0 && a->softcap >= 0.0f && a->d_q && a->d_k && a->d_v && a->d_q_gamma && a->d_k_gamma &&
           a->d_k_cache && a->d_v_cache;
}

// Heads of a block and lanes of a key row for this shape; slices: 16-byte pieces per lane (0: rows too wide)
struct Shape { int hb, lpk, slices, chunks; };
Shape shape_of(int wtype, int heads, int kv_heads, int dim, int vdim)
{
    const int e = wtype == B200_WT_F32 ? 4 : 8, n = (up8(dim) > up8(vdim) ? up8(dim) : up8(vdim)) / e, group = heads / kv_heads;
    Shape s = {};
    s.lpk = n <= 8 ? 8 : n <= 16 ? 16 : 32;
    s.slices = n <= 32 ? 1 : n <= 64 ? 2 : n <= 128 ? 4 : 0;
    if (!s.slices) return s;
    s.hb = 1;
    while (s.hb < group && s.hb < 4 / s.slices) s.hb <<= 1;
    s.chunks = (group + s.hb - 1) / s.hb;
    return s;
}

bool use_mma(int wtype, int dim, int vdim) { return wtype == B200_WT_BF16 && dim <= 256 && vdim <= 256; }

// Blocks of a cluster: no more than the cache has shares of a batch or two for
int cluster_of(int max_seq)
{
    int c = 1;
    while (c < MAX_CLUSTER && c * 128 <= max_seq) c <<= 1;
    return c;
}

// A launch of clusters, chained to the previous one when the caller asks for it
template <typename K, typename... Args>
int launch_clusters(K kern, const b200_gqa_args &a, int chunks, size_t smem, cudaStream_t st, Args... args)
{
    const int rc = allow_smem(kern, smem), cl = cluster_of(a.max_seq);
    if (rc) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.n_split * cl, a.kv_heads * chunks);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = cl; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.use_pdl ? 2 : 1;
    ++g_b200_launches;
    return (int)cudaLaunchKernelEx(&cfg, kern, a, cl, chunks, args...);
}

template <int DV>
int decode_mma(const b200_gqa_args &a, cudaStream_t st)
{
    const int group = a.heads / a.kv_heads, nh = group < MAX_HEADS ? group : MAX_HEADS, dqs = (a.dim + 15) / 16 * 16 + 8;
    auto bytes = [&](int stages) {
        const size_t tiles = (size_t)WARPS * stages * TK * (dqs + DV + 8) * 2, results = (size_t)WARPS * nh * up8(a.vdim) * 4;
        return ((size_t)TK * dqs + dqs + DV + 8) * 2 + ((size_t)nh * up8(a.vdim) + MAX_CLUSTER) * 4 + (tiles > results ? tiles : results);
    };
    const int stages = bytes(2) <= 220 * 1024 ? 2 : 1;
    return launch_clusters(gqa_decode_mma_kernel<DV>, a, (group + MAX_HEADS - 1) / MAX_HEADS, bytes(stages), st, dqs, stages);
}

template <int WT, int HB, int NS, int LPK>
int decode(const b200_gqa_args &a, const Shape &sp, cudaStream_t st)
{
    constexpr int NG = THREADS / LPK;
    const size_t smem = ((size_t)(NG + 1) * HB * up8(a.vdim) + HB * NG + MAX_CLUSTER) * 4 + (size_t)DEPTH * 4 * 2 * THREADS * 16;      // U * NS = 4
    return launch_clusters(gqa_decode_kernel<WT, HB, NS, LPK>, a, sp.chunks, smem, st);
}

template <int WT, int LPK>
int decode_narrow(const b200_gqa_args &a, const Shape &s, cudaStream_t st)
{
    return s.hb == 1 ? decode<WT, 1, 1, LPK>(a, s, st) : s.hb == 2 ? decode<WT, 2, 1, LPK>(a, s, st) : decode<WT, 4, 1, LPK>(a, s, st);
}

template <int WT>
int decode(const b200_gqa_args &a, cudaStream_t st)
{
    if (use_mma(WT, a.dim, a.vdim))
        return a.vdim <= 32 ? decode_mma<32>(a, st) : a.vdim <= 64 ? decode_mma<64>(a, st) : a.vdim <= 128 ? decode_mma<128>(a, st) : decode_mma<256>(a, st);
    const Shape s = shape_of(WT, a.heads, a.kv_heads, a.dim, a.vdim);
    switch (s.slices) {
    case 1: return s.lpk == 8 ? decode_narrow<WT, 8>(a, s, st) : s.lpk == 16 ? decode_narrow<WT, 16>(a, s, st) : decode_narrow<WT, 32>(a, s, st);
    case 2: return s.hb == 1 ? decode<WT, 1, 2, 32>(a, s, st) : decode<WT, 2, 2, 32>(a, s, st);
    case 4: return decode<WT, 1, 4, 32>(a, s, st);
    default: return B200_E_TOOLARGE;
    }
}

bool rows_ok(const b200_gqa_args *a)
{
    return shape_ok(a) && a->n_rows > 0 && a->pos0 >= 0 && a->pos0 + a->n_rows <= a->max_seq && a->proj_ld > 0 && a->d_q_rows;
}

}  // namespace

extern "C" int b200_gqa_splits(int wtype, int heads, int kv_heads, int dim, int vdim, int max_seq)
{
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || max_seq <= 0) return 1;
    const Shape s = shape_of(wtype, heads, kv_heads, dim, vdim);
    const int group = heads / kv_heads, chunks = use_mma(wtype, dim, vdim) ? (group + MAX_HEADS - 1) / MAX_HEADS : s.chunks > 0 ? s.chunks : 1;
    const int cl = cluster_of(max_seq), most = (max_seq + cl * BLOCK_KEYS - 1) / (cl * BLOCK_KEYS);
    int n = 148 / (kv_heads * chunks * cl);
    if (n > most) n = most;
    if (n > MAX_SPLITS) n = MAX_SPLITS;
    return n < 1 ? 1 : n;
}

extern "C" int b200_gqa_decode(const b200_gqa_args *a, void *stream)
{
    if (!shape_ok(a) || !a->d_part || !a->d_tickets || !a->d_out || !a->d_pos || a->n_split < 1 || a->n_split > MAX_SPLITS) return B200_E_BADARG;
    return a->wtype == B200_WT_BF16 ? decode<B200_WT_BF16>(*a, (cudaStream_t)stream) : decode<B200_WT_F32>(*a, (cudaStream_t)stream);
}

extern "C" int b200_gqa_rows_prep(const b200_gqa_args *a, void *stream)
{
    if (!rows_ok(a)) return B200_E_BADARG;
    cudaStream_t st = (cudaStream_t)stream;
    const int n = a->heads + 2 * a->kv_heads;
    const dim3 grid(a->n_rows, n > 4 * WARPS ? 2 : 1);
    if (a->wtype == B200_WT_BF16) gqa_prep_kernel<B200_WT_BF16><<<grid, THREADS, 0, st>>>(*a);
    else gqa_prep_kernel<B200_WT_F32><<<grid, THREADS, 0, st>>>(*a);
    ++g_b200_launches;
    return (int)cudaGetLastError();
}

extern "C" int b200_gqa_rows_attend(const b200_gqa_args *a, void *stream)
{
    if (!rows_ok(a) || !a->d_out_rows || a->out_ld < (long long)a->heads * a->vdim) return B200_E_BADARG;
    RowAttn r = {};
    r.n_rows = a->n_rows; r.pos0 = a->pos0; r.heads = a->heads; r.group = a->heads / a->kv_heads;
    r.dim = a->dim; r.vdim = a->vdim; r.scale = a->scale; r.softcap = a->softcap;
    r.q = a->d_q_rows;
    r.k = a->d_k_cache; r.k_ld = up8(a->dim); r.k_head = (long long)a->max_seq * r.k_ld;
    r.v = a->d_v_cache; r.v_ld = up8(a->vdim); r.v_head = (long long)a->max_seq * r.v_ld;
    r.k2 = a->d_k_cache;                                     // never read: there is no second part
    r.out = a->d_out_rows; r.out_ld = a->out_ld;
    cudaStream_t st = (cudaStream_t)stream;
    if (a->wtype == B200_WT_F32) return row_attend_f32(r, st);
    if (((uintptr_t)a->d_k_cache & 15) || ((uintptr_t)a->d_v_cache & 15) || ((uintptr_t)a->d_q_rows & 15)) return B200_E_BADARG;
    return a->softcap > 0.0f ? row_attend_bf16<true>(r, st) : row_attend_bf16<false>(r, st);
}
