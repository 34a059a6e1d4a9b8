// Attention over the paged cache for one step's queries, any mixture of prompt
// portions and single decoded tokens.
//
// A work item is (entry, a run of nq consecutive query tokens of that entry, one
// slice of the key range).  One block takes one item and one group of query heads
// that share a KV head, so the K/V pages are read once for all those rows
// (rows = nq tokens x gq heads).  Scores, the running maximum and sum of the
// streaming softmax and the output accumulator are 32-bit; the math per row is
//   s_j = (q . k_j) / sqrt(head_dim),  j in (pos - window, pos],  softmax,  sum_j w_j v_j
// as in the reference's compute_attention (src/model.cpp:1000-1052) and its paged
// form (src/paged_attention.cpp:11-90), without the 1e-9 guard in the divisor.
// Options for other designs, all off by default: the scale is an argument; with a
// window, the first keep_first keys of a request stay visible to every later query
// (at their true positions); a per-head penalty a_h * ln(1 + b_h * (pos - j)) is
// taken off the score of key j; values may have another head size than keys (a page
// is then [nkv][page_size][hd] keys followed by [nkv][page_size][hd_v] values); the
// scaled score may be capped, s <- c tanh(s / c), before a per-head slope times the
// distance, slope_h (pos - j), is taken off it; and the softmax may have a sink, a
// silent key without a value, of score 0 or of a learned score per head that is not
// scaled: w_j = exp(s_j) / (exp(sink_h) + sum_j exp(s_j)).  The sink enters as the
// starting state (maximum sink_h, sum 1) of the item's first key slice, so sliced
// items merge as they are.
// The window may stand still (`chunked`): a query at pos then sees the keys of its own chunk of W positions, counted
// from position 0.  Query rows may be wide (`wide`): a row has one block of lanes per KV head, the score of key j is the
// sum over the KV heads of block . that head's key (queries mixed across heads, see rope_store.cu), while its values are
// still those of the row's own KV head.  A gate per (token, head) may multiply the result (`out_gate`).  Key rows may be as
// wide as shared memory has room for; values wider than a block's threads hold are dealt to further blocks (grid z).
// The gate may be per output lane (`gate_lanes`).  A page may hold key rows alone (`one_row`): the values are the first hd_v
// lanes of the key rows.  And where rows are wide because one shared row is kept in blocks (`blocks`: attention over latent
// rows wider than a tile), the KV heads are those blocks, every query head meets all of them, and nh counts (block, query
// head) pairs, block after block: pair (G, h) has the wide row of query head h and sums the values of block G.  Results
// lie query head by query head, its blocks side by side.
// Items whose key range is sliced write (max, sum, unnormalised output) partials,
// merged by attn_merge_kernel in slice order.
#include "common.cuh"

#include <math_constants.h>

namespace {

constexpr int TK = 128;       // keys per tile = threads per block
constexpr int ITEM_INTS = 6;  // entry, q0, nq, slice, nslices, decode index

struct AttnArgs {
    const void* q;
    void* out;
    const void* pages;
    long long page_stride;
    const int* block_table;
    const int* table_row;  // entry -> row of block_table (a request's slot), or null: row = entry
    int max_blocks;
    const int* q_start;
    const int* q_len;
    const int* ctx_len;
    const int* items;
    float* part_o;
    float* part_ml;
    int nh, nkv, hd, page_size, num_pages, window;
    float scale;
    int* status;
    // bounds of the partial-result buffers, for callers whose buffers have a fixed size (0: not checked): decoded
    // tokens and key slices that part_o / part_ml were laid out for
    int part_tokens, part_slices;
    // the options: kept first keys, distance penalty per head (null: none), value head size
    int keep_first;
    const float* dist_a;
    const float* dist_b;
    int hd_v;
    // further options: scores capped as c tanh(s / c) (0: no cap); slope_h * (pos - j) taken off the score of key j
    // (null: none); a silent extra key of score 0 and no value in every softmax (its weight is lost)
    float softcap;
    const float* slope;
    int sink;
    const float* sink_value;    // with a sink: its score per head (null: 0); it is not scaled
    int chunked;                // the window is the chunk of `window` positions that pos lies in
    int wide;                   // q rows are [nkv][hd] lanes, one block per KV head
    const float* out_gate;      // [tokens][query heads] or null: what the result of a (token, head) is multiplied by
    int gate_lanes;             // out_gate is laid out as the result, a factor per lane
    int one_row;                // pages hold keys only: values are the first hd_v lanes of the key rows
    int blocks;                 // the KV heads are blocks of one shared row (see above)
};

template <typename T> struct Vec8;
template <> struct Vec8<float> {
    static __device__ __forceinline__ void load(const float* p, float (&f)[8]) {
        const float4 a = *reinterpret_cast<const float4*>(p);
        const float4 b = *reinterpret_cast<const float4*>(p + 4);
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
};
template <> struct Vec8<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&f)[8]) {
        const uint4 u = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            f[2 * i] = __uint_as_float(w[i] << 16);
            f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
};

// the first key a query at `pos` sees (kept first keys aside)
__device__ __forceinline__ int first_key(int pos, int W, int chunked) {
    if (W <= 0) return 0;
    return max(0, chunked ? pos - pos % W : pos - W + 1);
}

template <typename T, int RMAX>
__global__ __launch_bounds__(TK) void attn_paged_kernel(AttnArgs a) {
    extern __shared__ float smem[];
    const int hd = a.hd;
    const int qw = a.wide ? a.nkv * hd : hd;
    float* q_s = smem;                      // [RMAX][qw], pre-scaled
    float* p_s = q_s + RMAX * qw;           // [RMAX][TK]
    float* m_s = p_s + RMAX * TK;           // [RMAX] running maximum
    float* l_s = m_s + RMAX;                // [RMAX] running sum
    float* al_s = l_s + RMAX;               // [RMAX] rescale factor of the current tile
    float* da_s = al_s + RMAX;              // [RMAX] distance penalty of the row's head: a, b
    float* db_s = da_s + RMAX;
    int* lo_s = reinterpret_cast<int*>(db_s + RMAX);   // [RMAX] first key of the row's window
    long long* voff_s = reinterpret_cast<long long*>(lo_s + RMAX);  // [TK] element offset of each key's V row

    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int* item = a.items + (size_t)blockIdx.x * ITEM_INTS;
    const int e = item[0], q0 = item[1], slice = item[3], nslices = item[4], dec_index = item[5];
    const int qlen = a.q_len[e], ctx = a.ctx_len[e];
    // an item of a captured step is laid out for the largest portion the step serves: fewer tokens may be there
    const int nq = min(item[2], qlen - q0);
    if (a.part_tokens > 0 &&
        (dec_index < 0 || dec_index >= a.part_tokens || slice < 0 || slice >= nslices || nslices != a.part_slices)) {
        // the item's partial row would lie outside the fixed buffer: report it and touch nothing
        if (tid == 0) atomicOr(a.status, VCB_STATUS_BAD_ITEM);
        return;
    }

    const int g = a.nh / a.nkv;
    const int gq_max = g < RMAX ? g : RMAX;
    const int hchunks = (g + gq_max - 1) / gq_max;
    const int kvh = blockIdx.y / hchunks, hc = blockIdx.y % hchunks;
    const int head0 = kvh * g + hc * gq_max;
    const int gq = min(gq_max, g - hc * gq_max);
    if (qlen <= 0 || ctx <= 0 || nq <= 0) {
        // an empty entry: its slices still say "nothing here" (max = -inf, sum = 0), so that the merge writes zeros
        // rather than whatever the partial buffers held before
        if (nslices > 1 && a.part_ml != nullptr && tid < gq) {
            const int oh = a.blocks ? (head0 - kvh * g + tid) * a.nkv + kvh : head0 + tid;
            const size_t prow = ((size_t)dec_index * a.nh + oh) * nslices + slice;
            a.part_ml[prow * 2] = -CUDART_INF_F;
            a.part_ml[prow * 2 + 1] = 0.f;
        }
        return;
    }
    const int R = nq * gq;  // rows in use: r = iq * gq + ih
    // query heads, the first one here, and where head ih's result lies among a token's
    const int nqh = a.blocks ? g : a.nh, qh0 = a.blocks ? head0 - kvh * g : head0;
    auto out_head = [&](int ih) { return a.blocks ? (qh0 + ih) * a.nkv + kvh : head0 + ih; };

    const int row0 = a.q_start[e] + q0;       // flat token index of the first query
    const int pos0 = ctx - qlen + q0;         // its position
    const int pos_last = pos0 + nq - 1;
    const int W = a.window;

    // key range of the whole item, then of this slice (in pages)
    const int lo = first_key(pos0, W, a.chunked);
    const int hi = pos_last + 1;
    const int ps = a.page_size;
    const int pb_lo = lo / ps, pb_hi = (hi + ps - 1) / ps;
    const int pps = (pb_hi - pb_lo + nslices - 1) / nslices;
    const int my_pb_lo = pb_lo + slice * pps, my_pb_hi = min(pb_hi, my_pb_lo + pps);
    const int k_begin = max(lo, my_pb_lo * ps), k_end = min(hi, my_pb_hi * ps);
    // kept first keys that lie before the item's window: the first slice reads them ahead of its own range
    const int KF = W > 0 ? a.keep_first : 0;
    const int n_first = slice == 0 ? min(KF, lo) : 0;
    const int n_keys = n_first + max(0, k_end - k_begin);
    const int hdv = a.hd_v;
    const bool vec_ok = (hd % 8) == 0;

    // queries -> shared memory, scaled
    const T* qg = reinterpret_cast<const T*>(a.q);
    for (int idx = tid; idx < R * qw; idx += TK) {
        const int r = idx / qw, d = idx % qw;
        const int iq = r / gq, ih = r % gq;
        q_s[r * qw + d] = to_f32(qg[((size_t)(row0 + iq) * nqh + qh0 + ih) * qw + d]) * a.scale;
    }
    if (tid < RMAX) {
        const bool with_sink = a.sink && slice == 0;
        const int h = qh0 + tid % gq;
        m_s[tid] = with_sink ? (a.sink_value != nullptr && tid < R ? a.sink_value[h] : 0.f) : -CUDART_INF_F;
        l_s[tid] = with_sink ? 1.f : 0.f;
        da_s[tid] = a.dist_a != nullptr && tid < R ? a.dist_a[h] : (a.slope != nullptr && tid < R ? a.slope[h] : 0.f);
        db_s[tid] = a.dist_a != nullptr && tid < R ? a.dist_b[h] : 0.f;
        lo_s[tid] = first_key(pos0 + tid / gq, W, a.chunked);
    }
    constexpr int DPT = VCB_MAX_HEAD_DIM / TK;  // output dims per thread
    const int d0 = blockIdx.z * VCB_MAX_HEAD_DIM;   // first output dim of this block
    float acc_o[RMAX][DPT];
#pragma unroll
    for (int r = 0; r < RMAX; ++r)
#pragma unroll
        for (int i = 0; i < DPT; ++i) acc_o[r][i] = 0.f;
    __syncthreads();

    const T* pages = reinterpret_cast<const T*>(a.pages);
    const int* bt = a.block_table + (size_t)(a.table_row ? a.table_row[e] : e) * a.max_blocks;

    for (int u0 = 0; u0 < n_keys; u0 += TK) {
        const int n_valid = min(TK, n_keys - u0);
        // ---- phase 1: one key per thread, scores of all rows ----
        {
            const int u = u0 + tid;
            const int kidx = u < n_first ? u : k_begin + (u - n_first);
            float s[RMAX];
#pragma unroll
            for (int r = 0; r < RMAX; ++r) s[r] = 0.f;
            bool valid = tid < n_valid;
            if (valid) {
                const int page = bt[kidx / ps];
                if (page < 0 || page >= a.num_pages) {
                    atomicOr(a.status, VCB_STATUS_BAD_PAGE);
                    valid = false;
                    voff_s[tid] = -1;
                } else {
                    voff_s[tid] = (long long)page * a.page_stride + (a.one_row ? ((long long)kvh * ps + kidx % ps) * hd
                                  : (long long)a.nkv * ps * hd + ((long long)kvh * ps + kidx % ps) * hdv);
                    for (int b = 0; b < (a.wide ? a.nkv : 1); ++b) {
                        const T* kp = pages + (long long)page * a.page_stride + ((long long)(a.wide ? b : kvh) * ps + kidx % ps) * hd;
                        const float* q_b = q_s + b * hd;
                        if (!vec_ok) {
                            // a head size that is no multiple of 8: element by element
                            for (int c = 0; c < hd; ++c) {
                                const float kf = to_f32(kp[c]);
#pragma unroll
                                for (int r = 0; r < RMAX; ++r)
                                    if (r < R) s[r] = fmaf(kf, q_b[r * qw + c], s[r]);
                            }
                        }
                        for (int c = 0; vec_ok && c < hd; c += 8) {
                            float kf[8];
                            Vec8<T>::load(kp + c, kf);
#pragma unroll
                            for (int r = 0; r < RMAX; ++r) {
                                if (r < R) {
                                    const float4 qa = *reinterpret_cast<const float4*>(q_b + r * qw + c);
                                    const float4 qb = *reinterpret_cast<const float4*>(q_b + r * qw + c + 4);
                                    s[r] = fmaf(kf[0], qa.x, s[r]); s[r] = fmaf(kf[1], qa.y, s[r]);
                                    s[r] = fmaf(kf[2], qa.z, s[r]); s[r] = fmaf(kf[3], qa.w, s[r]);
                                    s[r] = fmaf(kf[4], qb.x, s[r]); s[r] = fmaf(kf[5], qb.y, s[r]);
                                    s[r] = fmaf(kf[6], qb.z, s[r]); s[r] = fmaf(kf[7], qb.w, s[r]);
                                }
                            }
                        }
                    }
                }
            }
#pragma unroll
            for (int r = 0; r < RMAX; ++r) {
                if (r < R) {
                    const int pos = pos0 + r / gq;
                    const bool seen = valid && kidx <= pos && (kidx >= lo_s[r] || kidx < KF);
                    float sc = s[r];
                    if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
                    if (a.dist_a != nullptr && seen) sc -= da_s[r] * logf(1.f + db_s[r] * (float)(pos - kidx));
                    else if (a.slope != nullptr && seen) sc -= da_s[r] * (float)(pos - kidx);
                    p_s[r * TK + tid] = seen ? sc : -CUDART_INF_F;
                }
            }
        }
        __syncthreads();
        // ---- phase 2: streaming softmax, rows dealt to warps ----
        for (int r = warp; r < R; r += TK / 32) {
            float v[TK / 32];
            float mx = -CUDART_INF_F;
#pragma unroll
            for (int i = 0; i < TK / 32; ++i) {
                v[i] = p_s[r * TK + lane + 32 * i];
                mx = fmaxf(mx, v[i]);
            }
            mx = warp_max(mx);
            const float m_old = m_s[r];
            const float m_new = fmaxf(m_old, mx);
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < TK / 32; ++i) {
                const float p = (v[i] == -CUDART_INF_F) ? 0.f : expf(v[i] - m_new);
                p_s[r * TK + lane + 32 * i] = p;
                sum += p;
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float alpha = (m_old == -CUDART_INF_F) ? 0.f : expf(m_old - m_new);
                al_s[r] = alpha;
                m_s[r] = m_new;
                l_s[r] = l_s[r] * alpha + sum;
            }
        }
        __syncthreads();
        // ---- phase 3: output dims dealt to threads ----
#pragma unroll
        for (int i = 0; i < DPT; ++i) {
            const int d = d0 + tid + i * TK;
            if (d < hdv) {
#pragma unroll
                for (int r = 0; r < RMAX; ++r)
                    if (r < R) acc_o[r][i] *= al_s[r];
                for (int j = 0; j < n_valid; ++j) {
                    const long long vo = voff_s[j];
                    if (vo < 0) continue;
                    const float v = to_f32(pages[vo + d]);
#pragma unroll
                    for (int r = 0; r < RMAX; ++r)
                        if (r < R) acc_o[r][i] = fmaf(p_s[r * TK + j], v, acc_o[r][i]);
                }
            }
        }
        __syncthreads();
    }

    // ---- write out ----
    if (nslices == 1) {
        T* og = reinterpret_cast<T*>(a.out);
#pragma unroll
        for (int i = 0; i < DPT; ++i) {
            const int d = d0 + tid + i * TK;
            if (d < hdv) {
#pragma unroll
                for (int r = 0; r < RMAX; ++r) {
                    if (r < R) {
                        const float l = l_s[r];
                        const int iq = r / gq, ih = r % gq;
                        const size_t row = (size_t)(row0 + iq) * a.nh + out_head(ih);
                        float o = l > 0.f ? acc_o[r][i] / l : 0.f;
                        if (a.out_gate != nullptr) o *= a.out_gate[a.gate_lanes ? row * hdv + d : (size_t)(row0 + iq) * nqh + qh0 + ih];
                        og[row * hdv + d] = from_f32<T>(o);
                    }
                }
            }
        }
    } else {
        // decode items only (nq == 1): partial row = (decode index, head, slice)
#pragma unroll
        for (int r = 0; r < RMAX; ++r) {
            if (r < R) {
                const size_t prow = ((size_t)dec_index * a.nh + out_head(r)) * nslices + slice;
#pragma unroll
                for (int i = 0; i < DPT; ++i) {
                    const int d = d0 + tid + i * TK;
                    if (d < hdv) a.part_o[prow * hdv + d] = acc_o[r][i];
                }
                if (tid == 0 && blockIdx.z == 0) {
                    a.part_ml[prow * 2] = m_s[r];
                    a.part_ml[prow * 2 + 1] = l_s[r];
                }
            }
        }
    }
}

// merge the slices of sliced items: grid (decode tokens, heads)
template <typename T>
__global__ void attn_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml,
                                  const int* __restrict__ dec_rows, T* __restrict__ out, int nh, int hd, int nslices,
                                  const float* __restrict__ out_gate, int gate_lanes, int gate_blocks) {
    pdl_trigger();
    pdl_wait();
    const int n = blockIdx.x, h = blockIdx.y;
    const size_t prow0 = ((size_t)n * nh + h) * nslices;
    // the slices' weights first (a batch of them at a time), each needed by every thread; then the outputs, several loads
    // in flight
    constexpr int MS = 64;
    __shared__ float w_s[MS], l_s[MS], m_all;
    if (threadIdx.x < 32) {
        float m = -CUDART_INF_F;
        for (int s = threadIdx.x; s < nslices; s += 32) m = fmaxf(m, part_ml[(prow0 + s) * 2]);
        m = warp_max(m);
        if (threadIdx.x == 0) m_all = m;
    }
    const int row = dec_rows[n];
    // (gate_blocks results side by side belong to one head)
    const float gate = out_gate != nullptr && !gate_lanes && row >= 0 ? out_gate[((size_t)row * nh + h) / gate_blocks] : 1.f;
    constexpr int DPT = 4;      // value lanes a thread (of blocks of 64 to 256 threads)
    for (int d0 = 0; d0 < hd; d0 += DPT * blockDim.x) {
        float l = 0.f, o[DPT] = {0.f, 0.f, 0.f, 0.f};
        for (int s0 = 0; s0 < nslices; s0 += MS) {
            const int ns = min(MS, nslices - s0);
            __syncthreads();
            if (threadIdx.x < ns) {
                const float ms = part_ml[(prow0 + s0 + threadIdx.x) * 2];
                const float w = ms == -CUDART_INF_F ? 0.f : expf(ms - m_all);
                w_s[threadIdx.x] = w;
                l_s[threadIdx.x] = ms == -CUDART_INF_F ? 0.f : part_ml[(prow0 + s0 + threadIdx.x) * 2 + 1] * w;
            }
            __syncthreads();
            for (int s = 0; s < ns; ++s) l += l_s[s];
#pragma unroll
            for (int k = 0; k < DPT; ++k) {
                const int d = d0 + threadIdx.x + k * blockDim.x;
                if (d < hd) {
                    const float* p = part_o + (prow0 + s0) * hd + d;
#pragma unroll 8
                    for (int s = 0; s < ns; ++s) {
                        const float w = w_s[s], x = p[(size_t)s * hd];
                        if (w != 0.f) o[k] = fmaf(x, w, o[k]);      // (a slice without keys may have left nothing)
                    }
                }
            }
        }
        if (row >= 0) {
#pragma unroll
            for (int k = 0; k < DPT; ++k) {
                const int d = d0 + threadIdx.x + k * blockDim.x;
                if (d < hd) {
                    const size_t at = ((size_t)row * nh + h) * hd + d;
                    out[at] = from_f32<T>((l > 0.f ? o[k] / l : 0.f) * (gate_lanes && out_gate != nullptr ? out_gate[at] : gate));
                }
            }
        }
    }
}

template <typename T, int RMAX>
int launch_attn(const AttnArgs& a, int n_items, cudaStream_t stream) {
    const int g = a.nh / a.nkv;
    const int gq_max = g < RMAX ? g : RMAX;
    const int hchunks = (g + gq_max - 1) / gq_max;
    const size_t qw = a.wide ? (size_t)a.nkv * a.hd : (size_t)a.hd;
    const int zblocks = (a.hd_v + VCB_MAX_HEAD_DIM - 1) / VCB_MAX_HEAD_DIM;
    const size_t smem = ((size_t)RMAX * qw + (size_t)RMAX * TK + 6 * RMAX) * sizeof(float) + TK * sizeof(long long);
    VCB_CHECK_ARG(smem <= 227 * 1024, "attn_paged: %d rows of %zu query lanes are more than a block's shared memory holds", RMAX, qw);
    auto kern = attn_paged_kernel<T, RMAX>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) {
            vcb_set_error("attn_paged: %zu bytes of shared memory refused: %s", smem, cudaGetErrorString(e));
            return -2;
        }
    }
    kern<<<dim3(n_items, a.nkv * hchunks, zblocks), TK, smem, stream>>>(a);
    VCB_CHECK_LAUNCH("attn_paged");
    return 0;
}

}  // namespace

// rows_max: 8 for items of single decoded tokens (key range may be sliced), 32 for prompt portions
// keep_first, dist_a / dist_b (float [nh] each, or null) and hd_v (0: as hd): the options named at the top of this file.
// chunked, wide, out_gate: likewise.  With them the key head size may be any number; values likewise.
VCB_API int vcb_attn_paged_ex(const void* q, void* out, int dtype, const void* pages, long long page_stride,
                              const int* block_table, const int* table_row, int max_blocks, const int* q_start, const int* q_len,
                              const int* ctx_len, const int* items, int n_items, int rows_max, float* part_o,
                              float* part_ml, int nh, int nkv, int hd, int page_size, int num_pages, int window,
                              float scale, int keep_first, const float* dist_a, const float* dist_b, int hd_v,
                              float softcap, const float* slope, int sink, const float* sink_value, int chunked, int wide,
                              const float* out_gate, int gate_lanes, int one_row, int blocks, int* status, cudaStream_t stream) {
    if (n_items == 0) return 0;
    if (hd_v <= 0) hd_v = hd;
    VCB_CHECK_ARG(!one_row || hd_v <= hd, "attn_paged: values of %d lanes in key rows of %d", hd_v, hd);
    VCB_CHECK_ARG(!blocks || (wide && dist_a == nullptr && slope == nullptr), "attn_paged: blocks of one shared row want wide query rows and no distance terms");
    VCB_CHECK_ARG(nh > 0 && nkv > 0 && nh % nkv == 0, "attn_paged: %d query heads are not a multiple of %d KV heads", nh, nkv);
    VCB_CHECK_ARG(hd >= 1 && hd_v >= 1, "attn_paged: head sizes %d (keys) and %d (values)", hd, hd_v);
    VCB_CHECK_ARG(hd % 8 != 0 || (page_stride % 8 == 0 && ((long long)nkv * page_size * hd) % 8 == 0),
                  "attn_paged: pages whose keys do not start on 8 elements (stride %lld)", page_stride);
    VCB_CHECK_ARG(rows_max == 8 || rows_max == 32, "attn_paged: rows_max must be 8 or 32");
    VCB_CHECK_ARG(page_size > 0 && window >= 0 && keep_first >= 0, "attn_paged: bad page_size %d, window %d or keep_first %d", page_size, window, keep_first);
    VCB_CHECK_ARG((dist_a == nullptr) == (dist_b == nullptr), "attn_paged: the distance penalty needs both of its vectors");
    VCB_CHECK_ARG(dist_a == nullptr || slope == nullptr, "attn_paged: a logarithmic penalty and a slope at once");
    VCB_CHECK_ARG(softcap >= 0.f, "attn_paged: a negative cap");
    AttnArgs a{q, out, pages, page_stride, block_table, table_row, max_blocks, q_start, q_len, ctx_len, items, part_o, part_ml,
               nh, nkv, hd, page_size, num_pages, window, scale, status, 0, 0, keep_first, dist_a, dist_b, hd_v,
               softcap, slope, sink, sink_value, chunked, wide, out_gate, gate_lanes, one_row, blocks};
    if (dtype == VCB_F32) return rows_max == 8 ? launch_attn<float, 8>(a, n_items, stream) : launch_attn<float, 32>(a, n_items, stream);
    return rows_max == 8 ? launch_attn<__nv_bfloat16, 8>(a, n_items, stream) : launch_attn<__nv_bfloat16, 32>(a, n_items, stream);
}

VCB_API int vcb_attn_paged(const void* q, void* out, int dtype, const void* pages, long long page_stride,
                           const int* block_table, const int* table_row, int max_blocks, const int* q_start, const int* q_len,
                           const int* ctx_len, const int* items, int n_items, int rows_max, float* part_o,
                           float* part_ml, int nh, int nkv, int hd, int page_size, int num_pages, int window,
                           float scale, int* status, cudaStream_t stream) {
    if (n_items == 0) return 0;
    VCB_CHECK_ARG(nh > 0 && nkv > 0 && nh % nkv == 0, "attn_paged: %d query heads are not a multiple of %d KV heads", nh, nkv);
    VCB_CHECK_ARG(hd >= 16 && hd % 16 == 0 && hd <= VCB_MAX_HEAD_DIM, "attn_paged: head_dim %d must be a multiple of 16 in [16, %d]", hd, VCB_MAX_HEAD_DIM);
    VCB_CHECK_ARG(rows_max == 8 || rows_max == 32, "attn_paged: rows_max must be 8 or 32");
    VCB_CHECK_ARG(page_size > 0 && window >= 0, "attn_paged: bad page_size %d or window %d", page_size, window);
    AttnArgs a{q, out, pages, page_stride, block_table, table_row, max_blocks, q_start, q_len, ctx_len, items, part_o, part_ml,
               nh, nkv, hd, page_size, num_pages, window, scale, status, 0, 0, 0, nullptr, nullptr, hd};
    if (dtype == VCB_F32) return rows_max == 8 ? launch_attn<float, 8>(a, n_items, stream) : launch_attn<float, 32>(a, n_items, stream);
    return rows_max == 8 ? launch_attn<__nv_bfloat16, 8>(a, n_items, stream) : launch_attn<__nv_bfloat16, 32>(a, n_items, stream);
}

VCB_API int vcb_attn_merge(const float* part_o, const float* part_ml, const int* dec_rows, void* out, int dtype,
                           int n_dec, int nh, int hd, int nslices, const float* out_gate, int gate_lanes, int gate_blocks, cudaStream_t stream) {
    if (n_dec == 0) return 0;
    const int threads = hd <= 64 ? 64 : (hd <= 128 ? 128 : 256);
    if (dtype == VCB_F32)
        launch_pdl(attn_merge_kernel<float>, dim3(n_dec, nh), dim3(threads), 0, stream, part_o, part_ml, dec_rows, (float*)out, nh, hd, nslices, out_gate, gate_lanes, gate_blocks);
    else
        launch_pdl(attn_merge_kernel<__nv_bfloat16>, dim3(n_dec, nh), dim3(threads), 0, stream, part_o, part_ml, dec_rows, (__nv_bfloat16*)out, nh, hd, nslices, out_gate, gate_lanes, gate_blocks);
    VCB_CHECK_LAUNCH("attn_merge");
    return 0;
}

// ---------------------------------------------------------------------------
// Sliced decode attention that allocates nothing (declared in no_alloc_api.h).
//
// Same kernels as vcb_attn_paged + vcb_attn_merge, but the (max, sum, output) partials of the key slices live in
// a fixed array inside this library instead of buffers the caller allocates.  The array exists once per GPU that
// loads the library, from load until exit, whether or not this entry point is ever called.
// ---------------------------------------------------------------------------
#include "no_alloc_api.h"

#include <mutex>

static __device__ __align__(256) float g_decode_partials[VCB_NO_ALLOC_SCRATCH_FLOATS];

namespace {
constexpr int MAX_DEVICES = 64;
float* g_partials_addr[MAX_DEVICES];   // device address of g_decode_partials on each device, once looked up
bool g_partials_known[MAX_DEVICES];
std::mutex g_partials_mutex;

// In host code `g_decode_partials` is only a handle for the runtime; the address a kernel can use must be asked
// for, per device, with that device current.
int partials_address(float** out) {
    int dev = -1;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess || dev < 0 || dev >= MAX_DEVICES) {
        vcb_set_error("attn_decode_no_alloc: cannot tell the current device (%s)", cudaGetErrorString(e));
        return -2;
    }
    std::lock_guard<std::mutex> lock(g_partials_mutex);
    if (!g_partials_known[dev]) {
        void* p = nullptr;
        e = cudaGetSymbolAddress(&p, g_decode_partials);
        if (e != cudaSuccess || p == nullptr) {
            vcb_set_error("attn_decode_no_alloc: cudaGetSymbolAddress failed on device %d: %s", dev, cudaGetErrorString(e));
            return -2;
        }
        g_partials_addr[dev] = static_cast<float*>(p);
        g_partials_known[dev] = true;
    }
    *out = g_partials_addr[dev];
    return 0;
}
}  // namespace

VCB_API int vcb_attn_decode_no_alloc(const void* q, void* out, int dtype, const void* pages, long long page_stride,
                                     const int* block_table, const int* table_row, int max_blocks,
                                     const int* q_start, const int* q_len, const int* ctx_len, const int* items,
                                     const int* dec_rows, int n_dec, int nslices, int nh, int nkv, int hd,
                                     int page_size, int num_pages, int window, float scale, int* status,
                                     cudaStream_t stream) {
    if (n_dec == 0) return 0;
    VCB_CHECK_ARG(n_dec > 0 && nslices >= 2, "attn_decode_no_alloc: needs at least one token and two key slices (got %d, %d)", n_dec, nslices);
    VCB_CHECK_ARG(nh > 0 && nkv > 0 && nh % nkv == 0, "attn_decode_no_alloc: %d query heads are not a multiple of %d KV heads", nh, nkv);
    VCB_CHECK_ARG(hd >= 16 && hd % 16 == 0 && hd <= VCB_MAX_HEAD_DIM, "attn_decode_no_alloc: head_dim %d must be a multiple of 16 in [16, %d]", hd, VCB_MAX_HEAD_DIM);
    VCB_CHECK_ARG(page_size > 0 && window >= 0, "attn_decode_no_alloc: bad page_size %d or window %d", page_size, window);
    const long long rows = (long long)n_dec * nh * nslices;
    const long long need = rows * (hd + 2);
    VCB_CHECK_ARG(need <= (long long)VCB_NO_ALLOC_SCRATCH_FLOATS,
                  "attn_decode_no_alloc: %d tokens x %d heads x %d slices x (head_dim %d + 2) = %lld floats of partials exceed "
                  "the built-in scratch of %lld floats; use fewer slices or the allocating entry points",
                  n_dec, nh, nslices, hd, need, (long long)VCB_NO_ALLOC_SCRATCH_FLOATS);
    float* scratch = nullptr;
    if (int rc = partials_address(&scratch)) return rc;
    float* part_o = scratch;               // [rows, hd]
    float* part_ml = scratch + rows * hd;  // [rows, 2]
    // Every (token, head, slice) row is written by the block that owns it before the merge reads it -- an empty
    // slice and an entry without tokens write max = -inf, sum = 0 -- so nothing of an earlier call's contents is
    // read and nothing has to be cleared.  The one exception is an item the kernel refuses (see below): its rows
    // keep what they held, the status word says so, and the output of that token is not to be used.
    // The kernel checks every item against the layout the array was cut for (n_dec tokens, nslices slices): an item
    // naming a token or slice beyond it, or another slice count, sets VCB_STATUS_BAD_ITEM and writes nothing.
    VCB_CHECK_ARG(status != nullptr, "attn_decode_no_alloc: a status word is required (bad items are reported there)");
    AttnArgs a{q, out, pages, page_stride, block_table, table_row, max_blocks, q_start, q_len, ctx_len, items, part_o,
               part_ml, nh, nkv, hd, page_size, num_pages, window, scale, status, n_dec, nslices, 0, nullptr, nullptr, hd};
    const int rc = dtype == VCB_F32 ? launch_attn<float, 8>(a, n_dec * nslices, stream)
                                    : launch_attn<__nv_bfloat16, 8>(a, n_dec * nslices, stream);
    if (rc) return rc;
    const int threads = hd <= 64 ? 64 : (hd <= 128 ? 128 : 256);
    if (dtype == VCB_F32)
        launch_pdl(attn_merge_kernel<float>, dim3(n_dec, nh), dim3(threads), 0, stream, part_o, part_ml, dec_rows, (float*)out, nh, hd, nslices, (const float*)nullptr, 0, 1);
    else
        launch_pdl(attn_merge_kernel<__nv_bfloat16>, dim3(n_dec, nh), dim3(threads), 0, stream, part_o, part_ml, dec_rows, (__nv_bfloat16*)out, nh, hd, nslices, (const float*)nullptr, 0, 1);
    VCB_CHECK_LAUNCH("attn_decode_no_alloc merge");
    return 0;
}
