// The launches of the decayed sum (matrix_state.cuh), in a source of their own so that they compile beside the others.
#include "matrix_state.cuh"

int matrix_state::launch_decayed_sum(const MatrixStateArgs& a, int requests, int cb, int col_blocks, cudaStream_t s) {
    return launch_dk<MODE_DECAYED_SUM>(a, requests, cb, col_blocks, s);
}
