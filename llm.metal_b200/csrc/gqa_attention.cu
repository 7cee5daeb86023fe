// Grouped-query attention with normed queries and keys (sm_100a): heads of any size, a per-position query factor, an
// optional cap on the scores, key and value rows cached in bfloat16 or fp32.
//
// Decode, one launch: a block serves up to HB query heads of one key/value head over its share of the cached positions.
// A key row lies across a group of lanes, sixteen bytes each; every group keeps an online softmax of its own, with the
// rows of the next positions in flight, and the first rows are fetched before the kernel waits for its predecessor.
// The newest position's key and value come from the projection; the block that owns it stores them. Groups merge
// through shuffles and shared memory, blocks through partial records and a ticket: the last one to finish merges.
//
// Prompt portions: gqa_prep writes cache rows and query rows of all tokens, the attention is that of row_attention.cuh.
#include "row_attention.cuh"

namespace {

constexpr int MIN_KEYS = 64;       // cached positions worth a block of their own
constexpr int MAX_SPLITS = 256;
constexpr int THREADS = 256, WARPS = THREADS / 32;

__host__ __device__ __forceinline__ int part_stride(int vdim) { return up8(vdim) + 8; }

// Elements col .. col + E of a projection's vector of n; zeros past its end.
template <int E>
__device__ __forceinline__ void load_part(float (&x)[E], const float *v, int col, int n)
{
#pragma unroll
    for (int e = 0; e < E; ++e) x[e] = col + e < n ? v[col + e] : 0.0f;
}

template <typename T> __device__ __forceinline__ float rounded(float x) { return (float)(T)x; }

template <int WT, int HB, int NS>
__global__ void __launch_bounds__(THREADS) gqa_decode_kernel(const __grid_constant__ b200_gqa_args p, int lpk, int chunks)
{
    using El = Elem<WT>;
    using T = typename El::T;
    constexpr int E = El::E, U = 4 / NS;                     // positions of a group in flight
    extern __shared__ __align__(16) float sh[];              // [WARPS][HB][up8(vdim) + 2], then the splits' weights
    __shared__ int s_last;
    pdl_launch_dependents();
    const int pos = *p.d_pos;
    if (pos < 0 || pos >= p.max_seq) return;
    int per = (pos + p.n_split - 1) / p.n_split;
    if (per < MIN_KEYS) per = MIN_KEYS;
    const int active = pos > 0 ? (pos + per - 1) / per : 1, split = blockIdx.x;
    if (split >= active) return;
    const int k_lo = split * per, k_hi = min(k_lo + per, pos);

    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int gpw = 32 / lpk, kg = warp * gpw + lane / lpk, KG = WARPS * gpw, sl = lane % lpk;
    const int kvh = blockIdx.y / chunks, h_in0 = (blockIdx.y % chunks) * HB, group = p.heads / p.kv_heads;
    const int h0 = kvh * group + h_in0, nh = min(HB, group - h_in0);
    const int d8 = up8(p.dim), v8 = up8(p.vdim);
    const T *kc = static_cast<const T *>(p.d_k_cache) + (size_t)kvh * p.max_seq * d8;
    const T *vc = static_cast<const T *>(p.d_v_cache) + (size_t)kvh * p.max_seq * v8;

    uint4 kr[U][NS], vr[U][NS];
    auto fetch = [&](int j0) {                               // positions j0, j0 + KG, ...
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int j = j0 + u * KG;
#pragma unroll
            for (int s = 0; s < NS; ++s) {
                const int col = (sl + s * lpk) * E;
                kr[u][s] = j < k_hi && col < d8 ? *reinterpret_cast<const uint4 *>(kc + (size_t)j * d8 + col) : make_uint4(0, 0, 0, 0);
                vr[u][s] = j < k_hi && col < v8 ? *reinterpret_cast<const uint4 *>(vc + (size_t)j * v8 + col) : make_uint4(0, 0, 0, 0);
            }
        }
    };
    fetch(k_lo + kg);
    float gq[NS][E], gk[NS][E];
#pragma unroll
    for (int s = 0; s < NS; ++s) { load_part<E>(gq[s], p.d_q_gamma, (sl + s * lpk) * E, p.dim); load_part<E>(gk[s], p.d_k_gamma, (sl + s * lpk) * E, p.dim); }
    const float factor = p.scale * (p.d_q_scale ? p.d_q_scale[pos] : 1.0f);
    pdl_wait();

    auto norm = [&](float (&x)[NS][E], const float (&g)[NS][E], float f) {
        float ss = 0.0f;
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) ss = fmaf(x[s][e], x[s][e], ss);
        for (int o = 1; o < lpk; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = f / sqrtf(ss / (float)p.dim + p.eps);
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) x[s][e] = g[s][e] * (x[s][e] * inv);
    };
    float q[HB][NS][E];
#pragma unroll
    for (int i = 0; i < HB; ++i) {
#pragma unroll
        for (int s = 0; s < NS; ++s) load_part<E>(q[i][s], p.d_q + (size_t)(h0 + min(i, nh - 1)) * p.dim, (sl + s * lpk) * E, p.dim);
        norm(q[i], gq, factor);
    }

    float m[HB], l[HB], acc[HB][NS][E];
#pragma unroll
    for (int i = 0; i < HB; ++i) {
        m[i] = -INFINITY; l[i] = 0.0f;
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) acc[i][s][e] = 0.0f;
    }
    auto reduce = [&](float a) {                             // over the lanes of a key
        for (int o = 1; o < lpk; o <<= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        return a;
    };
    auto cap = [&](float s) { return p.softcap > 0.0f ? p.softcap * tanhf(s / p.softcap) : s; };

    // every group of a warp takes the same number of trips: the shuffles are warp-wide
    for (int j0 = k_lo; j0 < k_hi; j0 += U * KG) {
        uint4 kn[U][NS], vn[U][NS];
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int s = 0; s < NS; ++s) { kn[u][s] = kr[u][s]; vn[u][s] = vr[u][s]; }
        if (j0 + U * KG < k_hi) fetch(j0 + U * KG + kg);
#pragma unroll
        for (int i = 0; i < HB; ++i) {
            float s_u[U], mt = m[i];
#pragma unroll
            for (int u = 0; u < U; ++u) {
                float a = 0.0f;
#pragma unroll
                for (int s = 0; s < NS; ++s) a += El::dot(kn[u][s], q[i][s]);
                a = cap(reduce(a));
                s_u[u] = j0 + kg + u * KG < k_hi ? a : -INFINITY;
                mt = fmaxf(mt, s_u[u]);
            }
            const float base = mt == -INFINITY ? 0.0f : mt, corr = expf(m[i] - base);
            m[i] = mt;
            l[i] *= corr;
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) acc[i][s][e] *= corr;
#pragma unroll
            for (int u = 0; u < U; ++u) {
                const float w = expf(s_u[u] - base);
                l[i] += w;
#pragma unroll
                for (int s = 0; s < NS; ++s) {
                    float v[E];
                    El::unpack(vn[u][s], v);
#pragma unroll
                    for (int e = 0; e < E; ++e) acc[i][s][e] = fmaf(w, v[e], acc[i][s][e]);
                }
            }
        }
    }
    if (split == active - 1 && warp == 0) {                  // the newest position, by the first group; the others only shuffle along
        float kx[NS][E], vx[NS][E];
#pragma unroll
        for (int s = 0; s < NS; ++s) {
            load_part<E>(kx[s], p.d_k + (size_t)kvh * p.dim, (sl + s * lpk) * E, p.dim);
            load_part<E>(vx[s], p.d_v + (size_t)kvh * p.vdim, (sl + s * lpk) * E, p.vdim);
        }
        norm(kx, gk, 1.0f);
        const bool store = lane < lpk && h_in0 == 0;
        T *kd = static_cast<T *>(p.d_k_cache) + ((size_t)kvh * p.max_seq + pos) * d8, *vd = static_cast<T *>(p.d_v_cache) + ((size_t)kvh * p.max_seq + pos) * v8;
#pragma unroll
        for (int s = 0; s < NS; ++s)
#pragma unroll
            for (int e = 0; e < E; ++e) {                    // padding columns are zeros
                const int col = (sl + s * lpk) * E + e;
                kx[s][e] = rounded<T>(kx[s][e]);
                vx[s][e] = rounded<T>(vx[s][e]);
                if (store && col < d8) kd[col] = (T)kx[s][e];
                if (store && col < v8) vd[col] = (T)vx[s][e];
            }
#pragma unroll
        for (int i = 0; i < HB; ++i) {
            float a = 0.0f;
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) a = fmaf(kx[s][e], q[i][s][e], a);
            a = cap(reduce(a));
            if (lane >= lpk) a = -INFINITY;
            const float mt = fmaxf(m[i], a), base = mt == -INFINITY ? 0.0f : mt, corr = expf(m[i] - base), w = expf(a - base);
            m[i] = mt;
            l[i] = fmaf(l[i], corr, w);
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) acc[i][s][e] = fmaf(acc[i][s][e], corr, w * vx[s][e]);
        }
    }

    // groups of a warp, then the warps of the block
    const int RS = v8 + 2;                                   // a warp's record: sums, maximum, total
#pragma unroll
    for (int i = 0; i < HB; ++i) {
        for (int o = lpk; o < 32; o <<= 1) {
            const float mo = __shfl_xor_sync(0xffffffffu, m[i], o), lo = __shfl_xor_sync(0xffffffffu, l[i], o);
            const float mt = fmaxf(m[i], mo), base = mt == -INFINITY ? 0.0f : mt, ca = expf(m[i] - base), cb = expf(mo - base);
            m[i] = mt;
            l[i] = l[i] * ca + lo * cb;
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) acc[i][s][e] = acc[i][s][e] * ca + __shfl_xor_sync(0xffffffffu, acc[i][s][e], o) * cb;
        }
        float *rec = sh + (size_t)(warp * HB + i) * RS;
        if (lane < lpk) {
#pragma unroll
            for (int s = 0; s < NS; ++s)
#pragma unroll
                for (int e = 0; e < E; ++e) {
                    const int col = (sl + s * lpk) * E + e;
                    if (col < v8) rec[col] = acc[i][s][e];
                }
            if (lane == 0) { rec[v8] = m[i]; rec[v8 + 1] = l[i]; }
        }
    }
    __syncthreads();
    const int PS = part_stride(p.vdim);
    for (int e = tid; e < nh * v8; e += THREADS) {
        const int i = e / v8, col = e % v8;
        float mt = -INFINITY;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) mt = fmaxf(mt, sh[(size_t)(w * HB + i) * RS + v8]);
        float a = 0.0f, t = 0.0f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float *rec = sh + (size_t)(w * HB + i) * RS;
            const float f = expf(rec[v8] - mt);              // a warp without keys weighs zero; the block has at least one
            a = fmaf(f, rec[col], a);
            t = fmaf(f, rec[v8 + 1], t);
        }
        if (active == 1) {
            if (col < p.vdim) p.d_out[(size_t)(h0 + i) * p.vdim + col] = a / t;
        } else {
            float *part = p.d_part + ((size_t)(h0 + i) * p.n_split + split) * PS;
            part[col] = a;
            if (col == 0) { part[v8] = mt; part[v8 + 1] = t; }
        }
    }
    if (active == 1) return;
    __threadfence();
    __syncthreads();
    if (tid == 0) s_last = atomicAdd(p.d_tickets + blockIdx.y, 1u) == (unsigned)active - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    if (tid == 0) p.d_tickets[blockIdx.y] = 0u;
    float *sw = sh;                                          // [HB][n_split]: the records have been read
    for (int i = warp; i < nh; i += WARPS) {
        const float *part = p.d_part + (size_t)(h0 + i) * p.n_split * PS;
        float mt = -INFINITY, t = 0.0f, ms[MAX_SPLITS / 32], ls[MAX_SPLITS / 32];
#pragma unroll
        for (int k = 0; k < MAX_SPLITS / 32; ++k) {
            const int s = lane + 32 * k;
            ms[k] = s < active ? __ldcg(part + (size_t)s * PS + v8) : -INFINITY;
            ls[k] = s < active ? __ldcg(part + (size_t)s * PS + v8 + 1) : 0.0f;
            mt = fmaxf(mt, ms[k]);
        }
        mt = warp_max(mt);
#pragma unroll
        for (int k = 0; k < MAX_SPLITS / 32; ++k) { ms[k] = expf(ms[k] - mt); t = fmaf(ms[k], ls[k], t); }
        t = warp_sum(t);
#pragma unroll
        for (int k = 0; k < MAX_SPLITS / 32; ++k)
            if (lane + 32 * k < active) sw[i * MAX_SPLITS + lane + 32 * k] = ms[k] / t;
    }
    __syncthreads();
    for (int e = tid; e < nh * p.vdim; e += THREADS) {
        const int i = e / p.vdim, col = e % p.vdim;
        const float *part = p.d_part + (size_t)(h0 + i) * p.n_split * PS + col;
        float a = 0.0f;
#pragma unroll 16
        for (int s = 0; s < active; ++s) a = fmaf(sw[i * MAX_SPLITS + s], __ldcg(part + (size_t)s * PS), a);
        p.d_out[(size_t)(h0 + i) * p.vdim + col] = a;
    }
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
            held[k] = e < n ? x[e] : 0.0f;
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
            if (e < n8) out[e] = (T)(e < n ? gamma[e] * (held[k] * inv) : 0.0f);
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
    s.lpk = 1;
    while (s.lpk < 32 && s.lpk < n) s.lpk <<= 1;
    s.slices = n <= s.lpk ? 1 : n <= 2 * s.lpk ? 2 : n <= 4 * s.lpk ? 4 : 0;
    if (!s.slices) return s;
    s.hb = 1;
    while (s.hb < group && s.hb < 4 / s.slices) s.hb <<= 1;
    s.chunks = (group + s.hb - 1) / s.hb;
    return s;
}

template <int WT, int HB, int NS>
int decode(const b200_gqa_args &a, const Shape &sp, cudaStream_t st)
{
    auto kern = gqa_decode_kernel<WT, HB, NS>;
    size_t smem = (size_t)WARPS * HB * (up8(a.vdim) + 2) * 4;
    if (smem < (size_t)HB * MAX_SPLITS * 4) smem = (size_t)HB * MAX_SPLITS * 4;
    const int rc = allow_smem(kern, smem);
    if (rc) return rc;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.n_split, a.kv_heads * sp.chunks);
    cfg.blockDim = dim3(THREADS);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = a.use_pdl ? 1 : 0;
    ++g_b200_launches;
    return (int)cudaLaunchKernelEx(&cfg, kern, a, sp.lpk, sp.chunks);
}

template <int WT>
int decode(const b200_gqa_args &a, cudaStream_t st)
{
    const Shape s = shape_of(WT, a.heads, a.kv_heads, a.dim, a.vdim);
    switch (s.slices * 10 + s.hb) {
    case 11: return decode<WT, 1, 1>(a, s, st);
    case 12: return decode<WT, 2, 1>(a, s, st);
    case 14: return decode<WT, 4, 1>(a, s, st);
    case 21: return decode<WT, 1, 2>(a, s, st);
    case 22: return decode<WT, 2, 2>(a, s, st);
    case 41: return decode<WT, 1, 4>(a, s, st);
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
    int n = 148 / (kv_heads * (s.chunks > 0 ? s.chunks : 1));
    const int most = (max_seq + MIN_KEYS - 1) / MIN_KEYS;
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
