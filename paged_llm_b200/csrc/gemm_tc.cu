// The many-token tcgen05 product (gemm_tc_duo.cuh: pairs of blocks on tiles of 256 tokens x 256 features).
#include "gemm_tc_duo.cuh"

// Waits inside the kernel that gave up since the library was loaded (0 unless something is broken).
PL_EXPORT int pl_gemm_tc_timeouts() {
    int n = 0;
    if (cudaMemcpyFromSymbol(&n, tc::g_timeouts, sizeof(int)) != cudaSuccess) return -1;
    return n;
}

// epi: 0 bfloat16 out, 1 float32 out, 2 SiLU (W = [Wg; Wu] of shape [2I, K], N = I outputs), 3 add (resid[M, N] +=,
// N a multiple of 4).  K a multiple of 64; rows of X and Y 16-byte aligned.
PL_EXPORT int pl_gemm_tc(const void* X, int ldx, const void* W, void* Y, int ldy, float* resid, int M, int N, int K, int epi,
                         cudaStream_t stream) {
    return gemm_tc_duo_launch(X, ldx, W, Y, ldy, resid, M, N, K, epi, stream);
}

// The same with an activation: act 0 SiLU, 1 the tanh form of GELU of a gate (W = [Wg; Wu]); 3: Y = relu(X W^T)^2.
PL_EXPORT int pl_gemm_tc_act(const void* X, int ldx, const void* W, void* Y, int ldy, int M, int N, int K, int act,
                             cudaStream_t stream) {
    return gemm_tc_duo_launch(X, ldx, W, Y, ldy, nullptr, M, N, K, act == 3 ? TC_BF16 : TC_SILU, stream, act);
}

// Grouped: X [cap, K] holds rows sorted by expert in tiles of 256 (tile i belongs to expert tile_expert[i], *n_tiles
// tiles are in use), W is [experts][N (or 2N for epilogue 2)][K]; Y [cap, ldy] in the order of X.  epi 0 (with act 3: the
// square of relu), 1 or 2.
PL_EXPORT int pl_gemm_tc_grouped(const void* X, int ldx, const void* W, void* Y, int ldy, int cap, int N, int K, int epi,
                                 int act, float act_limit, int experts, const int* n_tiles, const int* tile_expert,
                                 cudaStream_t stream) {
    PL_REQUIRE(experts > 0, "gemm_tc_grouped: experts=%d", experts);
    return gemm_tc_duo_launch(X, ldx, W, Y, ldy, nullptr, cap, N, K, epi, stream, act, experts, n_tiles, tile_expert, act_limit);
}
