#include "block_ops.cuh"
#include "common.cuh"
namespace mynn {
bool dense_gemm_tc_supported(int, const DenseGemm &) { return false; }
int launch_dense_gemm_tc(cudaStream_t, int, const DenseGemm &) { return fail(MYNN_E_UNSUPPORTED, "not built"); }
}
