// Entry points of the recurrences on a matrix state per head (matrix_rnn.cuh; each form's kernels are compiled in a file of
// their own, matrix_rnn_*.cu), and
//
//  * head_norm_gate          every head of o divided by its root mean square, times a gain (shared by the heads, or of its
//                            own), times silu(gate) where there is a gate
#include "matrix_rnn.cuh"

using namespace vcb_rnn;

namespace {

// a warp a (token, head)
template <typename TOUT>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, Rows gate, int gate_col, const float* __restrict__ w, int w_stride, float eps,
                                      const int* __restrict__ q_start, const int* __restrict__ q_len, int E, int T, int H, int dv,
                                      TOUT* __restrict__ out) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    if (item >= (long long)T * H) return;
    const int t = (int)(item / H), h = (int)(item % H);
    const size_t base = (size_t)t * H * dv + (size_t)h * dv;
    if (entry_of_row(q_start, q_len, E, t) < 0) {
        for (int c = lane; c < dv; c += 32) out[base + c] = from_f32<TOUT>(0.f);
        return;
    }
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) ss = fmaf(o[base + c], o[base + c], ss);
    ss = warp_sum(ss);
    const float rstd = rsqrtf(ss / (float)dv + eps);
    for (int c = lane; c < dv; c += 32) {
        float v = o[base + c] * rstd * (w != nullptr ? w[h * w_stride + c] : 1.f);
        if (gate.p != nullptr) v *= silu_f(rows_at(gate, t, gate_col + h * dv + c));
        out[base + c] = from_f32<TOUT>(v);
    }
}

int sm_count() {
    static int n = 0;
    if (n == 0) {
        int dev = 0;
        cudaGetDevice(&dev);
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
    }
    return n;
}

}  // namespace

// mode 0: the gated delta rule; 1: the gated linear form; 2: the decayed form; 3: retention; 4: the wkv form (see matrix_rnn.cuh).
// u [S][T][ld] the projection's sums; x [T][ldx] the convolved rows (mode 0); z [zS][T][zld] the decay's sums (modes 2 and 4).
// The columns may lie in other row blocks of u's buffer (q, k and v as results of products of their own): they are offsets.
// state [slots][H][dv][d] (a value column's d rows in a run).  out [rows][H * dv] 32-bit, rows >= the entries' tokens.
// Entries of no tokens are left out.
VCB_API int vcb_matrix_rnn(int mode, const float* u, int S, long long s_stride, long long ld, const float* x, long long ldx,
                           int q_col, int k_col, int v_col, int b_col, int a_col, const float* dt_bias, const float* rate,
                           const float* f_bias, const float* lower, float* state, long long state_stride, const int* q_start,
                           const int* q_len, const int* slots, int E, int rows, int H, int G, int d, int dv, float* out,
                           const float* z, int zS, long long z_stride, long long zld, float inv_tau, const float* decay,
                           const int* ctx_len, const float* freq, int rot, int interleaved, const float* bonus, cudaStream_t stream) {
    if (E == 0) return 0;
    VCB_CHECK_ARG(mode >= 0 && mode <= 4, "matrix_rnn: unknown mode %d", mode);
    VCB_CHECK_ARG(mode != 2 || (z != nullptr && f_bias != nullptr), "matrix_rnn: the decayed form needs the decay's sums and bias");
    VCB_CHECK_ARG(mode != 4 || (z != nullptr && f_bias != nullptr && bonus != nullptr), "matrix_rnn: the wkv form needs the decay's sums and bias and the bonus");
    VCB_CHECK_ARG(mode != 3 || (decay != nullptr && ctx_len != nullptr && rot >= 0 && rot <= d && rot % 2 == 0 && (rot == 0 || freq != nullptr)),
                  "matrix_rnn: retention needs a decay per head, the entries' positions and %d <= %d turning lanes with their frequencies", rot, d);
    VCB_CHECK_ARG(d >= 1 && d <= 512, "matrix_rnn: %d state rows a head (1 to 512)", d);
    VCB_CHECK_ARG(H >= 1 && G >= 1 && H % G == 0 && dv >= 1, "matrix_rnn: bad sizes H=%d G=%d dv=%d", H, G, dv);
    VCB_CHECK_ARG(H <= 65535 && E <= 65535, "matrix_rnn: %d heads, %d entries", H, E);
    VCB_CHECK_ARG(ld < (1 << 26) && ldx < (1 << 26), "matrix_rnn: rows of %lld and %lld lanes", ld, ldx);
    const int R = d <= 64 ? 8 : 16;     // rows a thread keeps of a column
    int L = 1;                          // lanes that share a column
    while (L * R < d) L <<= 1;
    // one column a thread while that gives no more blocks than there are SMs (a long portion of one request), else two
    const long long blocks1 = (long long)((dv + WALKERS / L - 1) / (WALKERS / L)) * H * E;
    const int C = blocks1 <= sm_count() ? 1 : 2;
    const int CT = C * WALKERS / L, DP = L * R;
    const int TB = DP <= 256 ? 16 : 8;
    int dp_shift = 0, ct_shift = 0;
    while ((1 << dp_shift) < DP) ++dp_shift;
    while ((1 << ct_shift) < CT) ++ct_shift;
    RnnArgs a{Rows{u, S < 1 ? 1 : S, s_stride, ld}, x, ldx, q_col, k_col, v_col, b_col, a_col, dt_bias, rate, f_bias, lower, state,
              state_stride, q_start, q_len, slots, out, H, G, d, dv, L, TB, dp_shift, ct_shift,
              Rows{z, zS < 1 ? 1 : zS, z_stride, zld}, inv_tau, decay, ctx_len, freq, rot, interleaved, bonus};
    const size_t smem = (size_t)(2 * ((row_decay(mode) ? 3 : 2) * TB * DP + TB * CT + 2 * TB) + TB * (CT + 1)) * sizeof(float);
    const dim3 grid((dv + CT - 1) / CT, H, E);
    const bool split = rows > 4 * E;    // some entry has more than four tokens
    const int rc = mode == MODE_DELTA     ? rnn_run<MODE_DELTA>(a, R, C, split, grid, smem, stream)
                   : mode == MODE_GATED   ? rnn_run<MODE_GATED>(a, R, C, split, grid, smem, stream)
                   : mode == MODE_DECAYED ? rnn_run<MODE_DECAYED>(a, R, C, split, grid, smem, stream)
                   : mode == MODE_RETAIN  ? rnn_run<MODE_RETAIN>(a, R, C, split, grid, smem, stream)
                                          : rnn_run<MODE_WKV>(a, R, C, split, grid, smem, stream);
    if (rc != 0) return rc;
    VCB_CHECK_LAUNCH("matrix_rnn");
    return 0;
}

// o [T][H * dv] 32-bit; gate (or null) [S][T][ld] sums whose columns gate_col .. gate_col + H dv gate o through a SiLU; w: a gain of
// dv lanes per head, w_stride apart (0: one for all heads), or null;
// out [T][H * dv] of out_dtype (zeros in rows outside every entry).
VCB_API int vcb_head_norm_gate(const float* o, const float* gate, int S, long long s_stride, long long ld, int gate_col,
                               const float* w, int w_stride, float eps, const int* q_start, const int* q_len, int E, int T, int H, int dv,
                               void* out, int out_dtype, cudaStream_t stream) {
    if (T == 0 || H == 0) return 0;
    const long long items = (long long)T * H;
    const int warps = 8;
    const dim3 grid((unsigned)((items + warps - 1) / warps));
    Rows g{gate, S < 1 ? 1 : S, s_stride, ld};
    if (out_dtype == VCB_F32)
        launch_pdl(head_norm_gate_kernel<float>, grid, dim3(32 * warps), 0, stream, o, g, gate_col, w, w_stride, eps, q_start, q_len, E, T, H, dv, (float*)out);
    else
        launch_pdl(head_norm_gate_kernel<__nv_bfloat16>, grid, dim3(32 * warps), 0, stream, o, g, gate_col, w, w_stride, eps, q_start, q_len, E, T, H,
                   dv, (__nv_bfloat16*)out);
    VCB_CHECK_LAUNCH("head_norm_gate");
    return 0;
}
