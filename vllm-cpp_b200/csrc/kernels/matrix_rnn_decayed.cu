// The kernels of the decayed form (matrix_rnn.cuh).
#include "matrix_rnn.cuh"

template int vcb_rnn::rnn_run<vcb_rnn::MODE_DECAYED>(const vcb_rnn::RnnArgs&, int, int, bool, dim3, size_t, cudaStream_t);
