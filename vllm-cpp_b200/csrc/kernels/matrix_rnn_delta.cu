// The kernels of the gated delta rule (matrix_rnn.cuh).
#include "matrix_rnn.cuh"

template int vcb_rnn::rnn_run<vcb_rnn::MODE_DELTA>(const vcb_rnn::RnnArgs&, int, int, bool, dim3, size_t, cudaStream_t);
