// Latent attention (sm_100a): keys and values of all heads are linear maps of one cached low-rank vector.
//
// Decode, three launches chained by programmatic dependent launch:
//   latent_absorb  per head q_lat = scale * W_uk^T q (the weight slice of a block is in registers before the
//                  previous kernel has finished); one extra block normalises the new token's latent, rotates its
//                  key part and the queries, and writes the cache row
//   latent_scores  split-sequence attention in the latent space: a block takes 32 cache rows at a time for sixteen
//                  heads (bfloat16: tensor cores; fp32: four heads, CUDA cores), rows staged once in shared memory
//                  and used for the scores and for the weighted sum; partial (sum, maximum, total) records per split
//   latent_value   merges the splits of a head, applies W_uv and the output gate
//
// Prompt portions: latent_prep writes cache rows and rotated queries of all rows; keys and values are expanded
// by a product the caller runs; the attention over them is the tiled one of row_attention.cuh.
#include "row_attention.cuh"

namespace {

constexpr int KT = 32;             // cache rows per tile of the decode scores = lanes of a warp
constexpr int HB = 4;              // heads per block of the fp32 decode scores, two warps each
constexpr int HB_MMA = 16;         // heads per block of the bfloat16 decode scores: the rows of a tensor-core tile
constexpr int ABSORB_PASSES = 4;   // row passes whose weights a warp of latent_absorb holds in registers
constexpr int VALUE_ROWS = 16;     // value rows per block of latent_value, two per warp
constexpr int MAX_SPLITS = 256;

// Element i of a rotated vector v whose first `dims` elements turn pairwise by the angles in rope (cos, sin).
__device__ __forceinline__ float rotated(const float *v, int i, int dims, const float *rope)
{
    if (i >= dims) return v[i];
    const float c = rope[i & ~1], s = rope[(i & ~1) + 1];
    const float a = v[i & ~1], b = v[(i & ~1) + 1];
    return (i & 1) ? b * c + a * s : a * c - b * s;
}

// The cache row of one token, by all 256 threads of a block. `wait` runs before anything an earlier kernel of the
// same token wrote is read; norm weights and angles are fetched ahead of it. `red` holds >= 33 floats.
template <typename T, typename Wait>
__device__ __forceinline__ void write_cache_row(const b200_latent_args &p, const float *dkv, int pos, float *red, Wait wait)
{
    constexpr int HELD = 4;                                  // elements a thread keeps in registers: 1024 a block
    const int R = p.kv_rank, R8 = up8(R), rot8 = up8(p.rot_dim), tid = threadIdx.x;
    T *row = static_cast<T *>(p.d_cache) + (size_t)pos * (R8 + rot8);
    const float *rope = p.d_rope + (size_t)pos * p.rot_dims;
    float g[HELD], v[HELD];
#pragma unroll
    for (int k = 0; k < HELD; ++k) g[k] = tid + k * 256 < R ? p.d_dkv_gamma[tid + k * 256] : 0.0f;
    float c = 1.0f, s = 0.0f;
    if (tid < p.rot_dims) { c = rope[tid & ~1]; s = rope[(tid & ~1) + 1]; }
    wait();
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < HELD; ++k) { v[k] = tid + k * 256 < R ? dkv[tid + k * 256] : 0.0f; ss = fmaf(v[k], v[k], ss); }
    for (int i = tid + HELD * 256; i < R; i += 256) ss = fmaf(dkv[i], dkv[i], ss);
    if (tid < rot8) {
        float r = 0.0f;
        if (tid < p.rot_dims) {
            const float x = dkv[R + (tid & ~1)], y = dkv[R + (tid & ~1) + 1];
            r = (tid & 1) ? y * c + x * s : x * c - y * s;
        } else if (tid < p.rot_dim) r = dkv[R + tid];
        row[R8 + tid] = (T)r;
    }
    for (int i = tid + 256; i < rot8; i += 256) row[R8 + i] = (T)(i < p.rot_dim ? rotated(dkv + R, i, p.rot_dims, rope) : 0.0f);
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)R + p.eps);
#pragma unroll
    for (int k = 0; k < HELD; ++k)
        if (tid + k * 256 < R8) row[tid + k * 256] = (T)(g[k] * (v[k] * inv));
    for (int i = tid + HELD * 256; i < R8; i += 256) row[i] = (T)(i < R ? p.d_dkv_gamma[i] * (dkv[i] * inv) : 0.0f);
}

// ------------------------------------------------------------------------------------------------ decode
// The position changes between tokens only, never between the kernels of one token, so each kernel may read it (and
// everything that depends on it alone: angles, cache rows of earlier tokens) before it waits for its predecessor.

template <int WT>
__global__ void __launch_bounds__(256) latent_absorb_kernel(const __grid_constant__ b200_latent_args p, int chunks, int lpr)
{
    using El = Elem<WT>;
    using T = typename El::T;
    constexpr int E = El::E;
    __shared__ float red[33];
    pdl_launch_dependents();
    const int R = p.kv_rank, R8 = up8(R), rot8 = up8(p.rot_dim), CS = R8 + rot8, dq = p.dim + p.rot_dim;
    const int pos = *p.d_pos;
    const bool valid = pos >= 0 && pos < p.max_seq;
    if ((int)blockIdx.x == p.heads * chunks) {
        if (valid) write_cache_row<T>(p, p.d_dkv, pos, red, [] { pdl_wait(); });
        else pdl_wait();
        return;
    }
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x / chunks, chunk = blockIdx.x % chunks;
    const int dim8 = up8(p.dim), rpw = 32 / lpr, sl = lane % lpr;
    const int row0 = (chunk * ABSORB_PASSES * 8 + warp) * rpw + lane / lpr;      // pass k adds k * 8 * rpw
    const T *w0 = static_cast<const T *>(p.d_w_uk_t) + (size_t)h * R * dim8;
    uint4 w[ABSORB_PASSES];
#pragma unroll
    for (int k = 0; k < ABSORB_PASSES; ++k) {
        const int row = row0 + k * 8 * rpw;
        w[k] = row < R && sl * E < dim8 ? *reinterpret_cast<const uint4 *>(w0 + (size_t)row * dim8 + sl * E) : make_uint4(0, 0, 0, 0);
    }
    pdl_wait();
    const float *q = p.d_q + (size_t)h * dq;
    float x[E];
#pragma unroll
    for (int e = 0; e < E; ++e) x[e] = sl * E + e < p.dim ? q[sl * E + e] : 0.0f;
    // the head's first block also rotates its query and clears the padding columns of the latent part
    if (chunk == 0 && valid) {
        T *ql = static_cast<T *>(p.d_qlat) + (size_t)h * CS;
        const float *rope = p.d_rope + (size_t)pos * p.rot_dims;
        for (int i = threadIdx.x; i < rot8; i += 256) ql[R8 + i] = (T)(i < p.rot_dim ? p.scale * rotated(q + p.dim, i, p.rot_dims, rope) : 0.0f);
        if ((int)threadIdx.x < R8 - R) ql[R + threadIdx.x] = (T)0.0f;
    }
#pragma unroll
    for (int k = 0; k < ABSORB_PASSES; ++k) {
        const int row = row0 + k * 8 * rpw;
        float acc = El::dot(w[k], x);
        if (row < R)
            for (int d = (sl + lpr) * E; d < dim8; d += lpr * E) {               // heads wider than a warp's slices
                float y[E];
#pragma unroll
                for (int e = 0; e < E; ++e) y[e] = d + e < p.dim ? q[d + e] : 0.0f;
                acc += El::dot(*reinterpret_cast<const uint4 *>(w0 + (size_t)row * dim8 + d), y);
            }
        for (int o = 1; o < lpr; o <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (sl == 0 && row < R) static_cast<T *>(p.d_qlat)[(size_t)h * CS + row] = (T)(p.scale * acc);
    }
}

// fp32, on the CUDA cores. Two warps per head: warp 2i + f of head i scores the tile's keys 16 f .. 16 f + 15 (two lanes per key, every
// other slice each) and sums the columns of half f (slices f, f + 2, ... of 32) of the weighted rows.
template <int NCH>
__global__ void __launch_bounds__(256) latent_scores_f32_kernel(const __grid_constant__ b200_latent_args p, int row16)
{
    using El = Elem<B200_WT_F32>;
    using T = float;
    constexpr int E = El::E;
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float ssh[HB][KT];
    pdl_launch_dependents();
    const int R8 = up8(p.kv_rank), rot8 = up8(p.rot_dim), CS = R8 + rot8, PS = R8 + 8;
    const int S = CS / E;                                    // 16-byte slices of a cache row
    unsigned char *keys = smem;                              // [KT] rows, row16 slices apart (2 mod 4: no bank conflicts)
    float *qs = reinterpret_cast<float *>(smem + (size_t)KT * row16 * 16);       // [HB][CS]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, hi = warp >> 1, half = warp & 1;
    const int h0 = blockIdx.y * HB, h = h0 + hi, split = blockIdx.x;
    const int pos = *p.d_pos;
    const bool valid = pos >= 0 && pos < p.max_seq;
    const int lo = valid && p.window > 0 && pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
    const int nk = valid ? pos - lo + 1 : 0;
    const int tiles = (nk + KT - 1) / KT, per = (tiles + p.n_split - 1) / p.n_split;
    const int t0 = split * per, t1 = min(t0 + per, tiles);
    const T *cache = static_cast<const T *>(p.d_cache);

    // rows of a tile except the new token's, which this token's previous kernel has written
    auto stage_row = [&](int r, int kp) {
        for (int c = lane; c < S; c += 32) cp16(smem_u32(keys + ((size_t)r * row16 + c) * 16), cache + (size_t)kp * CS + (size_t)c * E, true);
    };
    auto stage = [&](int tile) {
        const int k0 = tile * KT, n = min(KT, nk - k0);
#pragma unroll
        for (int i = 0; i < KT / 8; ++i) {
            const int r = warp + 8 * i;
            if (r < n && lo + k0 + r != pos) stage_row(r, lo + k0 + r);
        }
    };
    if (t0 < t1) stage(t0);
    pdl_wait();
    {
        const int n = min(HB, p.heads - h0) * CS / 4;        // queries: contiguous fp32 rows
        for (int i = threadIdx.x; i < n; i += 256) cp16(smem_u32(qs + 4 * i), static_cast<const float *>(p.d_qlat) + (size_t)h0 * CS + 4 * i, true);
        if (t0 < t1 && t1 == tiles && warp == 0) {           // the newest key is the last row of the last tile
            const int r = nk - 1 - (tiles - 1) * KT;
            if (tiles - 1 == t0) stage_row(r, pos);
        }
    }
    float m = -INFINITY, l = 0.0f, acc[NCH][E];
#pragma unroll
    for (int c = 0; c < NCH; ++c)
#pragma unroll
        for (int e = 0; e < E; ++e) acc[c][e] = 0.0f;
    for (int tile = t0; tile < t1; ++tile) {
        if (tile > t0) {
            __syncthreads();
            stage(tile);
            if (tile == tiles - 1 && warp == 0) stage_row(nk - 1 - tile * KT, pos);
        }
        cp_commit();
        cp_wait<0>();
        __syncthreads();
        const int n = min(KT, nk - tile * KT);
        {
            const int k = half * 16 + (lane >> 1), par = lane & 1;
            float a = 0.0f, b = 0.0f;
            if (k < n && h < p.heads) {
                const uint4 *kr = reinterpret_cast<const uint4 *>(keys + (size_t)k * row16 * 16);
                const float *q = qs + (size_t)hi * CS;
                int c = par;
#pragma unroll 2
                for (; c + 2 < S; c += 4) { a += El::dot(kr[c], q + c * E); b += El::dot(kr[c + 2], q + (c + 2) * E); }
                if (c < S) a += El::dot(kr[c], q + c * E);
            }
            a += b;
            a += __shfl_xor_sync(0xffffffffu, a, 1);
            if (par == 0) ssh[hi][k] = k < n ? a : -INFINITY;
        }
        __syncthreads();
        const float s = ssh[hi][lane];
        const float mt = fmaxf(m, warp_max(s));
        const float w = lane < n ? expf(s - mt) : 0.0f;
        const float corr = m == -INFINITY ? 0.0f : expf(m - mt);
        l = l * corr + warp_sum(w);
        m = mt;
#pragma unroll
        for (int c = 0; c < NCH; ++c)
#pragma unroll
            for (int e = 0; e < E; ++e) acc[c][e] *= corr;
#pragma unroll 4
        for (int j = 0; j < n; ++j) {
            const float wj = __shfl_sync(0xffffffffu, w, j);
#pragma unroll
            for (int c = 0; c < NCH; ++c) {
                const int sl = (2 * c + half) * 32 + lane;
                if (sl * E < R8) {
                    float v[E];
                    El::unpack(*reinterpret_cast<const uint4 *>(keys + ((size_t)j * row16 + sl) * 16), v);
#pragma unroll
                    for (int e = 0; e < E; ++e) acc[c][e] = fmaf(wj, v[e], acc[c][e]);
                }
            }
        }
    }
    if (h >= p.heads) return;
    float *part = p.d_part + ((size_t)h * p.n_split + split) * PS;
#pragma unroll
    for (int c = 0; c < NCH; ++c) {
        const int col = ((2 * c + half) * 32 + lane) * E;
        if (col < R8)
#pragma unroll
            for (int e = 0; e < E; e += 4)
                *reinterpret_cast<float4 *>(part + col + e) = make_float4(acc[c][e], acc[c][e + 1], acc[c][e + 2], acc[c][e + 3]);
    }
    if (half == 0 && lane == 0) { part[R8] = m; part[R8 + 1] = l; }
}

// bfloat16, on the tensor cores: sixteen heads are the rows of both products, so a cache row is read from shared
// memory once per sixteen heads. Warp w scores keys 8 (w & 3) .. + 7 over half w >> 2 of the columns, keeps the
// softmax state of heads 2 w and 2 w + 1, and sums NTW tiles of eight latent columns of the weighted rows. Two tiles
// of keys in shared memory, the next one's copies under the current one.
template <int NTW>
__global__ void __launch_bounds__(256) latent_scores_bf16_kernel(const __grid_constant__ b200_latent_args p, int row16)
{
    constexpr int PST = KT + 8;                              // row of the weights in shared memory: 16 bytes off 64
    extern __shared__ __align__(16) unsigned char smem[];
    __shared__ float sc[2][HB_MMA][KT + 1], corr_sh[HB_MMA];
    __shared__ __align__(16) __nv_bfloat16 wsh[HB_MMA][PST];
    pdl_launch_dependents();
    const int R8 = up8(p.kv_rank), rot8 = up8(p.rot_dim), CS = R8 + rot8, PS = R8 + 8;
    const int S = CS / 8, SP = (S + 3) & ~3;                 // 16-byte slices of a row; padded to steps of 32 columns
    const uint32_t rowb = row16 * 16;                        // odd in 16-byte units: ldmatrix is conflict-free
    const uint32_t qs = smem_u32(smem), ks = qs + HB_MMA * rowb;          // [16] query rows, [2][KT] key rows
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h0 = blockIdx.y * HB_MMA, split = blockIdx.x;
    const int pos = *p.d_pos;
    const bool valid = pos >= 0 && pos < p.max_seq;
    const int lo = valid && p.window > 0 && pos - p.window + 1 > 0 ? pos - p.window + 1 : 0;
    const int nk = valid ? pos - lo + 1 : 0;
    const int tiles = (nk + KT - 1) / KT, per = (tiles + p.n_split - 1) / p.n_split;
    const int t0 = split * per, t1 = min(t0 + per, tiles);
    const __nv_bfloat16 *cache = static_cast<const __nv_bfloat16 *>(p.d_cache);

    auto copy_row = [&](uint32_t dst, const __nv_bfloat16 *src, bool on) {         // columns past the row hold zeros
        for (int c = lane; c < SP; c += 32) cp16(dst + c * 16, src + (c < S ? c * 8 : 0), on && c < S);
    };
    auto stage = [&](int tile) {                             // all rows but the new token's; rows past the last hold zeros
        const int k0 = lo + tile * KT;
#pragma unroll
        for (int i = 0; i < KT / 8; ++i) {
            const int r = warp + 8 * i, kp = k0 + r;
            if (kp != pos) copy_row(ks + ((tile & 1) * KT + r) * rowb, cache + (size_t)(kp < pos ? kp : 0) * CS, kp < pos);
        }
    };
    auto stage_newest = [&](int tile) {
        if (tile == tiles - 1 && warp == 0) copy_row(ks + ((tile & 1) * KT + nk - 1 - tile * KT) * rowb, cache + (size_t)pos * CS, true);
    };
    if (t0 < t1) stage(t0);
    pdl_wait();
    if (t0 < t1) {
        const __nv_bfloat16 *q = static_cast<const __nv_bfloat16 *>(p.d_qlat);
#pragma unroll
        for (int i = 0; i < HB_MMA / 8; ++i) {
            const int r = warp + 8 * i, h = h0 + r;
            copy_row(qs + r * rowb, q + (size_t)(h < p.heads ? h : 0) * CS, h < p.heads);
        }
        stage_newest(t0);
    }
    cp_commit();

    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f}, acc[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i)
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[i][k] = 0.0f;
    for (int tile = t0; tile < t1; ++tile) {
        if (tile + 1 < t1) {
            stage(tile + 1);
            stage_newest(tile + 1);
        }
        cp_commit();
        cp_wait<1>();
        __syncthreads();
        const uint32_t kt = ks + (tile & 1) * KT * rowb;
        {   // scores: 16 heads x 8 keys per warp, this half of the columns
            const int steps = SP / 4, mid = (steps + 1) / 2, s0 = warp < 4 ? 0 : mid, s1 = warp < 4 ? mid : steps;
            const uint32_t qa = qs + (lane & 15) * rowb + (lane >> 4) * 16;
            const uint32_t ka = kt + ((warp & 3) * 8 + (lane & 7)) * rowb + (lane >> 3) * 16;
            float d[2][4] = {{0.0f, 0.0f, 0.0f, 0.0f}, {0.0f, 0.0f, 0.0f, 0.0f}};
#pragma unroll 3
            for (int s = s0; s < s1; ++s) {                  // 32 columns
                uint32_t a[4], a2[4], b[4];
                ldsm4(qa + s * 64, a);
                ldsm4(qa + s * 64 + 32, a2);
                ldsm4(ka + s * 64, b);
                mma_bf16(d[0], a, b[0], b[1]);
                mma_bf16(d[1], a2, b[2], b[3]);
            }
            const int r = lane >> 2, c = (warp & 3) * 8 + (lane & 3) * 2;
#pragma unroll
            for (int k = 0; k < 4; ++k) sc[warp >> 2][r + (k >> 1) * 8][c + (k & 1)] = d[0][k] + d[1][k];
        }
        __syncthreads();
        const int n = nk - tile * KT;
#pragma unroll
        for (int i = 0; i < 2; ++i) {                        // a lane per key
            const int r = 2 * warp + i;
            const float s = lane < n ? sc[0][r][lane] + sc[1][r][lane] : -INFINITY;
            const float mt = fmaxf(m[i], warp_max(s));
            const float w = lane < n ? expf(s - mt) : 0.0f;
            const float corr = m[i] == -INFINITY ? 0.0f : expf(m[i] - mt);
            l[i] = fmaf(l[i], corr, warp_sum(w));
            m[i] = mt;
            wsh[r][lane] = __float2bfloat16_rn(w);
            if (lane == 0) corr_sh[r] = corr;
        }
        __syncthreads();
        const float c0 = corr_sh[lane >> 2], c1 = corr_sh[(lane >> 2) + 8];
        uint32_t wa[KT / 16][4];
#pragma unroll
        for (int k = 0; k < KT / 16; ++k) ldsm4(smem_u32(&wsh[lane & 15][k * 16 + (lane >> 4) * 8]), wa[k]);
#pragma unroll
        for (int i = 0; i < NTW; i += 2) {
            const int col = (warp * NTW + i) * 8;
            if (col >= R8) break;                            // uniform across the warp
#pragma unroll
            for (int j = 0; j < 2; ++j) { acc[i + j][0] *= c0; acc[i + j][1] *= c0; acc[i + j][2] *= c1; acc[i + j][3] *= c1; }
            const uint32_t va = kt + (lane & 15) * rowb + (col + (lane >> 4) * 8) * 2;
#pragma unroll
            for (int k = 0; k < KT / 16; ++k) {
                uint32_t b[4];
                ldsm4_t(va + k * 16 * rowb, b);
                mma_bf16(acc[i], wa[k], b[0], b[1]);
                mma_bf16(acc[i + 1], wa[k], b[2], b[3]);
            }
        }
        __syncthreads();                                     // this tile's rows, scores and weights are overwritten next
    }
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
        const int col = (warp * NTW + i) * 8 + (lane & 3) * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int h = h0 + (lane >> 2) + 8 * r;
            if (col < R8 && h < p.heads)
                *reinterpret_cast<float2 *>(p.d_part + ((size_t)h * p.n_split + split) * PS + col) = make_float2(acc[i][2 * r], acc[i][2 * r + 1]);
        }
    }
    if (lane < 2 && h0 + 2 * warp + lane < p.heads) {
        float *part = p.d_part + ((size_t)(h0 + 2 * warp + lane) * p.n_split + split) * PS;
        part[R8] = lane ? m[1] : m[0];
        part[R8 + 1] = lane ? l[1] : l[0];
    }
}

template <int WT>
__global__ void __launch_bounds__(256) latent_value_kernel(const __grid_constant__ b200_latent_args p, int chunks, int sgroups)
{
    using El = Elem<WT>;
    using T = typename El::T;
    constexpr int E = El::E, RPW = VALUE_ROWS / 8, NS = 2, BATCH = 16;
    extern __shared__ __align__(16) unsigned char smem[];
    float *olat = reinterpret_cast<float *>(smem);           // [sgroups][up8(kv_rank)]
    __shared__ float sw[MAX_SPLITS];
    pdl_launch_dependents();
    const int R8 = up8(p.kv_rank), PS = R8 + 8, S = R8 / E;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x / chunks, v0 = (blockIdx.x % chunks) * VALUE_ROWS + warp * RPW;
    const int dim8 = up8(p.dim), per_head = dim8 + up8(p.vdim);
    const T *w0 = static_cast<const T *>(p.d_w_kv) + ((size_t)h * per_head + dim8) * R8;
    uint4 w[RPW][NS];
#pragma unroll
    for (int k = 0; k < RPW; ++k)
#pragma unroll
        for (int s = 0; s < NS; ++s)
            w[k][s] = v0 + k < p.vdim && s * 32 + lane < S ? *reinterpret_cast<const uint4 *>(w0 + (size_t)(v0 + k) * R8 + (s * 32 + lane) * E)
                                                           : make_uint4(0, 0, 0, 0);
    pdl_wait();
    const float *part = p.d_part + (size_t)h * p.n_split * PS;
    const float gate = lane < RPW && v0 + lane < p.vdim ? p.d_gate[h * p.vdim + v0 + lane] : 0.0f;
    // A thread sums four columns over every sgroups-th split. Its first loads are in flight while warp 0 turns the
    // splits' maxima and totals into weights.
    const int cg = R8 / 4, col4 = (int)threadIdx.x % cg, sg = (int)threadIdx.x / cg;
    float4 held[BATCH];
    if (sg < sgroups)
#pragma unroll
        for (int i = 0; i < BATCH; ++i) {
            const int s = sg + i * sgroups;
            held[i] = s < p.n_split ? *reinterpret_cast<const float4 *>(part + (size_t)s * PS + 4 * col4) : make_float4(0, 0, 0, 0);
        }
    if (warp == 0) {
        float m = -INFINITY, l = 0.0f, ms[MAX_SPLITS / 32], ls[MAX_SPLITS / 32];
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; ++i) {
            const int s = lane + 32 * i;
            ms[i] = s < p.n_split ? part[(size_t)s * PS + R8] : -INFINITY;
            ls[i] = s < p.n_split ? part[(size_t)s * PS + R8 + 1] : 0.0f;
            m = fmaxf(m, ms[i]);
        }
        m = warp_max(m);
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; ++i) {
            ms[i] = ls[i] > 0.0f ? expf(ms[i] - m) : 0.0f;
            l = fmaf(ms[i], ls[i], l);
        }
        l = warp_sum(l);
        const float inv = l > 0.0f ? 1.0f / l : 0.0f;
#pragma unroll
        for (int i = 0; i < MAX_SPLITS / 32; ++i)
            if (lane + 32 * i < p.n_split) sw[lane + 32 * i] = ms[i] * inv;
    }
    __syncthreads();
    if (sg < sgroups)
        for (int c4 = col4; c4 < cg; c4 += 256) {            // a second trip only where a row is wider than 1024
            float4 a = make_float4(0, 0, 0, 0);
            int s = sg;
            if (c4 == col4) {
#pragma unroll
                for (int i = 0; i < BATCH; ++i, s += sgroups) {
                    const float f = s < p.n_split ? sw[s] : 0.0f;
                    a.x = fmaf(f, held[i].x, a.x); a.y = fmaf(f, held[i].y, a.y); a.z = fmaf(f, held[i].z, a.z); a.w = fmaf(f, held[i].w, a.w);
                }
            }
#pragma unroll 8
            for (; s < p.n_split; s += sgroups) {
                const float f = sw[s];
                const float4 v = *reinterpret_cast<const float4 *>(part + (size_t)s * PS + 4 * c4);
                a.x = fmaf(f, v.x, a.x); a.y = fmaf(f, v.y, a.y); a.z = fmaf(f, v.z, a.z); a.w = fmaf(f, v.w, a.w);
            }
            *reinterpret_cast<float4 *>(olat + (size_t)sg * R8 + 4 * c4) = a;
        }
    __syncthreads();
    if (sgroups > 1) {
        for (int r = threadIdx.x; r < R8; r += 256) {
            float a = olat[r];
            for (int g = 1; g < sgroups; ++g) a += olat[(size_t)g * R8 + r];
            olat[r] = a;                                     // this thread alone reads and writes column r
        }
        __syncthreads();
    }
    float y[RPW];
#pragma unroll
    for (int k = 0; k < RPW; ++k) y[k] = 0.0f;
#pragma unroll
    for (int s = 0; s < NS; ++s)
        if (s * 32 + lane < S) {
            float x[E];
#pragma unroll
            for (int e = 0; e < E; e += 4) *reinterpret_cast<float4 *>(x + e) = *reinterpret_cast<const float4 *>(olat + (s * 32 + lane) * E + e);
#pragma unroll
            for (int k = 0; k < RPW; ++k) y[k] += El::dot(w[k][s], x);
        }
    for (int c = NS * 32 + lane; c < S; c += 32)
#pragma unroll
        for (int k = 0; k < RPW; ++k)
            if (v0 + k < p.vdim) y[k] += El::dot(*reinterpret_cast<const uint4 *>(w0 + (size_t)(v0 + k) * R8 + (size_t)c * E), olat + c * E);
    float mine = 0.0f;
#pragma unroll
    for (int k = 0; k < RPW; ++k) {
        const float t = warp_sum(y[k]);
        if (lane == k) mine = t;
    }
    if (lane < RPW && v0 + lane < p.vdim) p.d_out[h * p.vdim + v0 + lane] = mine * sigmoid_f32(gate);
}

// ------------------------------------------------------------------------------------------------ rows

template <int WT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const __grid_constant__ b200_latent_args p)
{
    using T = typename Elem<WT>::T;
    __shared__ float red[33];
    const int m = blockIdx.x, pos = p.pos0 + m;
    write_cache_row<T>(p, p.d_dkv + (size_t)m * p.proj_ld, pos, red, [] {});
    const int dim8 = up8(p.dim), rot8 = up8(p.rot_dim), dq = p.dim + p.rot_dim, QS = dim8 + rot8;
    const float *q = p.d_q + (size_t)m * p.proj_ld;
    const float *rope = p.d_rope + (size_t)pos * p.rot_dims;
    T *out = static_cast<T *>(p.d_q_rows) + (size_t)m * p.heads * QS;
    // a warp per head, two elements (one rotated pair) per lane
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int h = warp; h < p.heads; h += 8) {
        const float *qh = q + (size_t)h * dq;
        for (int e = 2 * lane; e < QS; e += 64) {
            float v[2];
            if (e < dim8) {
                v[0] = e < p.dim ? qh[e] : 0.0f;
                v[1] = e + 1 < p.dim ? qh[e + 1] : 0.0f;
            } else {
                const int r = e - dim8;
                v[0] = r < p.rot_dim ? qh[p.dim + r] : 0.0f;
                v[1] = r + 1 < p.rot_dim ? qh[p.dim + r + 1] : 0.0f;
                if (r < p.rot_dims) {
                    const float c = rope[r], s = rope[r + 1], x = v[0], y = v[1];
                    v[0] = x * c - y * s;
                    v[1] = y * c + x * s;
                }
            }
            T *o = out + (size_t)h * QS + e;
            if constexpr (WT == B200_WT_BF16) *reinterpret_cast<__nv_bfloat162 *>(o) = __floats2bfloat162_rn(v[0], v[1]);
            else *reinterpret_cast<float2 *>(o) = make_float2(v[0], v[1]);
        }
    }
}

// ------------------------------------------------------------------------------------------------ host side

bool shape_ok(const b200_latent_args *a)
{
    return a && (a->wtype == B200_WT_BF16 || a->wtype == B200_WT_F32) && a->heads > 0 && a->dim > 0 && a->rot_dim > 0 && a->vdim > 0 &&
           a->kv_rank > 0 && a->max_seq > 0 && a->rot_dims >= 0 && a->rot_dims <= a->rot_dim && a->rot_dims % 2 == 0 &&
           a->d_q && a->d_dkv && a->d_dkv_gamma && a->d_rope && a->d_cache;
}

// 256 threads, chained to the previous launch when pdl is set
template <typename K, typename... Args>
int launch_pdl(K kern, int gx, int gy, size_t smem, int pdl, cudaStream_t st, Args... args)
{
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(gx, gy);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = smem;
    cfg.stream = st;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl ? 1 : 0;
    ++g_b200_launches;
    return (int)cudaLaunchKernelEx(&cfg, kern, args...);
}

template <int WT>
int decode(const b200_latent_args &a, cudaStream_t st)
{
    constexpr int E = Elem<WT>::E;
    const int dim8 = up8(a.dim), R8 = up8(a.kv_rank), CS = R8 + up8(a.rot_dim);
    int lpr = 1;
    while (lpr < 32 && lpr * E < dim8) lpr <<= 1;
    const int rows_per_block = ABSORB_PASSES * 8 * (32 / lpr);
    const int chunks = (a.kv_rank + rows_per_block - 1) / rows_per_block;
    int rc = launch_pdl(latent_absorb_kernel<WT>, a.heads * chunks + 1, 1, 0, a.use_pdl, st, a, chunks, lpr);
    if (rc) return rc;

#define SCORES(K, GROUPS)                                                                     \
    do {                                                                                      \
        if ((rc = allow_smem(K, smem)) != 0) return rc;                                        \
        rc = launch_pdl(K, a.n_split, GROUPS, smem, a.use_pdl, st, a, row16);                  \
    } while (0)
    if (WT == B200_WT_BF16) {
        int row16 = (CS / 8 + 3) & ~3;                       // steps of 32 columns, then odd
        row16 |= 1;
        const size_t smem = (size_t)(HB_MMA + 2 * KT) * row16 * 16;
        const int groups = (a.heads + HB_MMA - 1) / HB_MMA;
        if (R8 <= 128) SCORES(latent_scores_bf16_kernel<2>, groups);
        else if (R8 <= 256) SCORES(latent_scores_bf16_kernel<4>, groups);
        else if (R8 <= 512) SCORES(latent_scores_bf16_kernel<8>, groups);
        else if (R8 <= 1024) SCORES(latent_scores_bf16_kernel<16>, groups);
        else return B200_E_TOOLARGE;
    } else {
        int row16 = CS / E;                                  // 2 mod 4: four keys x two slices touch different banks
        while (row16 % 4 != 2) ++row16;
        const size_t smem = (size_t)KT * row16 * 16 + (size_t)HB * CS * 4;
        const int groups = (a.heads + HB - 1) / HB;
        if (R8 <= 64 * E) SCORES(latent_scores_f32_kernel<1>, groups);
        else if (R8 <= 128 * E) SCORES(latent_scores_f32_kernel<2>, groups);
        else if (R8 <= 256 * E) SCORES(latent_scores_f32_kernel<4>, groups);
        else return B200_E_TOOLARGE;
    }
#undef SCORES
    if (rc) return rc;
    const int vchunks = (a.vdim + VALUE_ROWS - 1) / VALUE_ROWS;
    const int sgroups = R8 / 4 >= 256 ? 1 : 256 / (R8 / 4) < a.n_split ? 256 / (R8 / 4) : a.n_split;
    return launch_pdl(latent_value_kernel<WT>, a.heads * vchunks, 1, (size_t)sgroups * R8 * 4, a.use_pdl, st, a, vchunks, sgroups);
}

// the tiled attention over rows: keys [W_uk c | rotated part], values W_uv c, all heads with rows of their own
RowAttn row_args(const b200_latent_args &a)
{
    const int dim8 = up8(a.dim), rot8 = up8(a.rot_dim), vd8 = up8(a.vdim), R8 = up8(a.kv_rank), es = a.wtype == B200_WT_F32 ? 4 : 2;
    RowAttn r = {};
    r.n_rows = a.n_rows; r.pos0 = a.pos0; r.heads = a.heads; r.group = 1; r.window = a.window;
    r.dim = a.dim; r.rot_dim = a.rot_dim; r.vdim = a.vdim; r.scale = a.scale;
    r.q = a.d_q_rows;
    r.k = a.d_kv; r.k_ld = a.kv_ld; r.k_head = dim8 + vd8; r.kv_row0 = a.kv_row0;
    r.v = static_cast<const char *>(a.d_kv) + (size_t)dim8 * es; r.v_ld = a.kv_ld; r.v_head = dim8 + vd8;
    r.k2 = static_cast<const char *>(a.d_cache) + (size_t)R8 * es; r.k2_ld = R8 + rot8;
    r.gate = a.d_gate; r.gate_ld = a.proj_ld;
    r.out = a.d_out_rows; r.out_ld = a.out_ld;
    return r;
}

}  // namespace

extern "C" int b200_latent_splits(int heads, int window, int max_seq)
{
    if (heads <= 0 || max_seq <= 0) return 1;
    const int span = window > 0 && window < max_seq ? window : max_seq;
    const int tiles = (span + KT - 1) / KT, groups = (heads + HB_MMA - 1) / HB_MMA;
    int n = 148 / groups;
    if (n > tiles) n = tiles;
    if (n > MAX_SPLITS) n = MAX_SPLITS;
    return n < 1 ? 1 : n;
}

extern "C" int b200_latent_decode(const b200_latent_args *a, void *stream)
{
    if (!shape_ok(a) || !a->d_gate || !a->d_w_uk_t || !a->d_w_kv || !a->d_qlat || !a->d_part || !a->d_out || !a->d_pos ||
        a->n_split < 1 || a->n_split > MAX_SPLITS)
        return B200_E_BADARG;
    return a->wtype == B200_WT_BF16 ? decode<B200_WT_BF16>(*a, (cudaStream_t)stream) : decode<B200_WT_F32>(*a, (cudaStream_t)stream);
}

static bool rows_ok(const b200_latent_args *a)
{
    return shape_ok(a) && a->n_rows > 0 && a->pos0 >= 0 && a->pos0 + a->n_rows <= a->max_seq && a->proj_ld > 0 && a->d_q_rows;
}

extern "C" int b200_latent_rows_prep(const b200_latent_args *a, void *stream)
{
    if (!rows_ok(a)) return B200_E_BADARG;
    cudaStream_t st = (cudaStream_t)stream;
    if (a->wtype == B200_WT_BF16) latent_prep_kernel<B200_WT_BF16><<<a->n_rows, 256, 0, st>>>(*a);
    else latent_prep_kernel<B200_WT_F32><<<a->n_rows, 256, 0, st>>>(*a);
    ++g_b200_launches;
    return (int)cudaGetLastError();
}

extern "C" int b200_latent_rows_attend(const b200_latent_args *a, void *stream)
{
    const int oldest = a && a->window > 0 && a->pos0 - a->window + 1 > 0 ? a->pos0 - a->window + 1 : 0;
    if (!rows_ok(a) || !a->d_gate || !a->d_kv || !a->d_out_rows || a->kv_row0 < 0 || a->kv_row0 > oldest ||
        a->kv_ld < (long long)a->heads * (up8(a->dim) + up8(a->vdim)) || a->out_ld < (long long)a->heads * a->vdim)
        return B200_E_BADARG;
    cudaStream_t st = (cudaStream_t)stream;
    if (a->wtype == B200_WT_BF16) {
        if ((a->kv_ld & 7) || ((uintptr_t)a->d_kv & 15) || ((uintptr_t)a->d_q_rows & 15)) return B200_E_BADARG;
        return row_attend_bf16<false>(row_args(*a), st);
    }
    return row_attend_f32(row_args(*a), st);
}
