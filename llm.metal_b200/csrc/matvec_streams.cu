// The BF16 and F32 instantiations of the kernel in matvec_core.cuh with layer norms, learned positions, residual streams
// and the squared relu.
#include "matvec_core.cuh"

int b200_mv::launch_streams(const b200_matvec_args &a, const Geometry &geo, int spt, int rb, int grid, cudaStream_t st)
{
    return launch_typed<FAM_STREAMS>(a, geo, spt, rb, grid, st);
}
