// The BF16 and F32 instantiations of the kernel in matvec_core.cuh (post-norm inputs, gated outputs, depth sums).
#include "matvec_core.cuh"

int b200_mv::launch_ext(const b200_matvec_args &a, const Geometry &geo, int spt, int rb, int grid, cudaStream_t st)
{
    if (a.wtype == B200_WT_BF16)
        return spt == 1 ? launch_by_rows<B200_WT_BF16, 1>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_BF16, 2>(a, geo, rb, grid, st);
    return spt == 1 ? launch_by_rows<B200_WT_F32, 1>(a, geo, rb, grid, st)
         : spt == 2 ? launch_by_rows<B200_WT_F32, 2>(a, geo, rb, grid, st) : launch_by_rows<B200_WT_F32, 4>(a, geo, rb, grid, st);
}
