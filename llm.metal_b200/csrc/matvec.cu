// b200_matvec: argument checks, launch geometry and the Q8_0 / F16 instantiations of the kernel in matvec_core.cuh.
#include "matvec_core.cuh"

#include <stdlib.h>

unsigned long long g_b200_launches = 0;

extern "C" unsigned long long b200_launch_count(int reset)
{
    unsigned long long v = g_b200_launches;
    if (reset) g_b200_launches = 0;
    return v;
}

extern "C" void b200_launch_count_add(unsigned long long n) { g_b200_launches += n; }

namespace {

int g_sm_count = 0;
int sm_count()
{
    if (!g_sm_count) {
        int dev = 0, n = 0;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0)
            n = 148;
        g_sm_count = n;
    }
    return g_sm_count;
}

// Tuning knobs from the environment, read once per process: consumer threads per block and the ring
// budget in KB (defaults measured on Qwen3-4B shapes).
struct Knobs { int group_threads, ring_kb; };
const Knobs &knobs()
{
    static const Knobs k = [] {
        auto env_int = [](const char *name, int dflt) { const char *e = getenv(name); return e && *e ? atoi(e) : dflt; };
        Knobs v;
        v.group_threads = env_int("LLMB200_MV_GROUP_THREADS", 640);
        v.ring_kb = env_int("LLMB200_MV_RING_KB", 192);
        return v;
    }();
    return k;
}

} // namespace

using namespace b200_mv;

extern "C" int b200_matvec(const b200_matvec_args *ap, void *stream)
{
    if (!ap) return B200_E_BADARG;
    const b200_matvec_args &a = *ap;
    if (!a.d_w || a.rows <= 0 || a.cols <= 0 || (a.row_stride % 16) || ((uintptr_t)a.d_w % 16)) return B200_E_BADARG;
    if (a.wtype < B200_WT_Q8 || a.wtype > B200_WT_F32) return B200_E_BADARG;
    const bool ext = a.wtype == B200_WT_BF16 || a.wtype == B200_WT_F32;
    if (a.wtype == B200_WT_Q8 ? (a.cols % 32) : (a.cols % 8)) return B200_E_BADARG;
    if (a.row_stride < (long long)b200_packed_row_stride(a.wtype, a.cols)) return B200_E_BADARG;
    if (a.in_mode == B200_IN_VEC ? !a.d_in_vec
        : a.in_mode == B200_IN_RESID ? (!a.d_resid_in || a.n_slots < 0 || (a.n_slots > 0 && !a.d_slots))
        : a.in_mode == B200_IN_POSTNORM ? (!ext || !a.d_in_vec || !a.d_slot_norm_gamma || (a.d_mix_in && !a.d_mix_coef))
        : a.in_mode == B200_IN_EMBED ? (!a.d_emb || !a.d_tokens || !a.d_pos || a.emb_rows <= 0) : true)
        return B200_E_BADARG;
    const bool streams = a.out_mode == B200_OUT_STREAMS || a.d_norm_beta || a.d_slot_norm_beta || a.d_emb_pos ||
                         (a.out_mode == B200_OUT_STORE && a.act == B200_ACT_RELU2);
    // one launch takes its optional parts from one family
    if (streams && (!ext || a.in_mode == B200_IN_POSTNORM || a.out_mode == B200_OUT_GATED || a.out_mode == B200_OUT_GLU || a.hist_n ||
                    a.softcap != 0.0f || (a.d_norm_gamma && !a.d_norm_beta)))
        return B200_E_BADARG;
    if (!ext && (a.out_mode == B200_OUT_GATED || a.norm_dim || a.norm_groups || a.hist_n || a.glu_rows || a.softcap != 0.0f)) return B200_E_BADARG;
    if (ext && (a.norm_dim < 0 || a.norm_dim > a.cols || a.norm_groups < 0 ||
                (a.norm_groups > 1 && (a.norm_dim > 0 ? a.norm_dim : a.cols) % a.norm_groups) ||
                a.hist_n < 0 || (a.hist_n > 0 && (!a.d_hist || !a.d_hist_coef || !a.d_hist_out)) ||
                (a.glu_rows && (a.out_mode != B200_OUT_GLU || a.glu_rows < 0 || a.glu_rows % 2 || a.glu_rows > a.rows || !a.d_out2)) ||
                (a.in_mode == B200_IN_RESID && a.d_slot_norm_gamma) || (a.d_norm_beta && (!a.d_norm_gamma || a.norm_groups > 1)) ||
                (a.d_slot_norm_beta && (a.in_mode != B200_IN_EMBED || !a.d_slot_norm_gamma)) ||
                (a.d_emb_pos && (a.in_mode != B200_IN_EMBED || a.emb_pos_rows < 1)) ||
                (a.out_mode == B200_OUT_STREAMS && (a.n_streams < 1 || a.n_streams > B200_MAX_STREAMS || !a.d_streams_in || !a.d_streams_out ||
                                                    !a.d_connect))))
        return B200_E_BADARG;
    if (a.out_mode == B200_OUT_GATED ? (!a.d_out[0] || !a.d_out_resid || !a.d_out_gate || !a.d_out_gate_bias)
        : a.out_mode == B200_OUT_STREAMS ? !a.d_out[0]
        : a.out_mode == B200_OUT_GLU ? (a.rows % 2 || !a.d_out[0]) : (a.out_mode != B200_OUT_STORE || a.n_out < 1 || a.n_out > B200_MAX_PEERS))
        return B200_E_BADARG;
    if (a.n_wait < 0 || a.n_wait > B200_MAX_PEERS || a.n_signal < 0 || a.n_signal > B200_MAX_PEERS ||
        a.n_argmax_out < 0 || a.n_argmax_out > B200_MAX_PEERS)
        return B200_E_BADARG;
    if ((a.n_wait > 0 || a.n_signal > 0) && (!a.d_epoch || !a.d_err)) return B200_E_BADARG;
    if ((a.n_signal > 0 || a.advance_pos || a.advance_epoch || a.d_next_token || a.d_argmax_scratch) && !a.d_ticket)
        return B200_E_BADARG;
    if ((a.advance_pos || a.d_next_token) && !a.d_pos_rw) return B200_E_BADARG;
    if (a.d_next_token && (!a.d_prompt_len || !a.d_argmax_scratch)) return B200_E_BADARG;
    if (a.advance_epoch && (!a.d_epoch || !a.d_epoch_rw)) return B200_E_BADARG;
    if (a.d_argmax_scratch && a.out_mode != B200_OUT_STORE) return B200_E_BADARG;

    const int E = a.wtype == B200_WT_Q8 ? 16 : a.wtype == B200_WT_F32 ? 4 : 8;
    const int nsl = (a.cols + E - 1) / E;
    // Up to two slices per thread: keeps a group at <= 320 threads for rows of up to 640 slices, so that
    // two blocks (this kernel's and the next one's) fit on an SM; 960 consumers + the producer warp at most.
    // Measured on the 2560 x 9728 down projection: two slices per thread 12.3 us, one slice 16.3 us.
    const int spt = nsl <= 320 ? 1 : a.wtype == B200_WT_F32 && nsl > 1920 ? 4 : 2;
    if ((nsl + spt - 1) / spt > 960) return B200_E_TOOLARGE;
    Geometry geo;
    geo.T = (((nsl + spt - 1) / spt) + 31) / 32 * 32;
    const int ralign = a.out_mode == B200_OUT_GLU ? 2 : 1;
    const int units = a.rows / ralign;

    // rows per stage: 16-24 KB per bulk copy
    int rb = 8;
    while (rb > 1 && (long long)rb * a.row_stride > 24576) rb >>= 1;
    if (rb < ralign) rb = ralign;
    geo.slot_bytes = (unsigned)(((long long)rb * a.row_stride + 127) / 128 * 128);
    geo.NG = knobs().group_threads / geo.T;
    if (geo.NG > 8) geo.NG = 8;
    if (geo.NG < 1) geo.NG = 1;
    // Ring slots: a multiple of the group count, so that a slot is always consumed by the same group.
    // A group works through its stages in order, hence never waits on a slot whose previous phase is
    // still open -- mbarrier parity waits cannot tell phase k from phase k-2.
    const int ring_budget = knobs().ring_kb * 1024;
    while (geo.NG > 1 && (long long)geo.NG * geo.slot_bytes > ring_budget) --geo.NG;
    int per_group = ring_budget / (int)(geo.NG * geo.slot_bytes);
    if (per_group < 1) per_group = 1;
    while (per_group > 1 && per_group * geo.NG > 12) --per_group;
    geo.nstage = per_group * geo.NG;
    geo.share_x = geo.NG > 1 && (a.in_mode != B200_IN_VEC || a.d_norm_gamma) && (size_t)spt * geo.T * E * 4 <= 16384;

    int grid = a.grid;
    if (grid <= 0) grid = sm_count();                // one block per SM
    if (grid > units) grid = units;
    cudaStream_t st = (cudaStream_t)stream;
    if (a.wtype == B200_WT_Q8)
        return spt == 1 ? launch_by_rows<B200_WT_Q8, 1>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_Q8, 2>(a, geo, rb, grid, st);
    if (streams) return launch_streams(a, geo, spt, rb, grid, st);
    if (ext) return launch_ext(a, geo, spt, rb, grid, st);
    return spt == 1 ? launch_by_rows<B200_WT_F16, 1>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_F16, 2>(a, geo, rb, grid, st);
}
