// Rotary attention whose options are all parameters: what lies between the stacked q, k, v projection and the attention
// kernels, and the turn back behind them.
//
//  * qkv_rope_store   from a token's 32-bit sums [q | k | v] (or [q | k], where the keys as projected double as values):
//                     optionally all query lanes divided by one root mean square and multiplied by a gain per lane, the
//                     key lanes likewise; the first `rot` lanes of every q and k head turned by position * freq[i], lanes
//                     paired in halves (i, i + rot/2) or interleaved (2i, 2i+1); optionally every value head turned the
//                     same way over `vrot` of its lanes with frequencies of its own; queries to a buffer, keys and values
//                     to the token's place in the paged cache.  Further options: a bias on every lane before all else;
//                     every value head divided by its root mean square; columns behind the projection that are one
//                     gate per query head or per lane of the heads' results (their sigmoids go to a buffer for the
//                     attention kernels' epilogues); queries mixed across heads on their way out, see below; and values
//                     mixed with those that an earlier layer made of the same token, v <- (1 - l) v + l v_first, l a
//                     learned number (that layer leaves its values, 32-bit, in a buffer of the step).
//
// Mixed queries: where the scores of the heads are mixed before the softmax, score_h <- sum_g T[h][g] (q_g . k_kv(g)), the sum
// over g can be drawn into the queries: with q'_h[G] = sum over the heads g that read KV head G of T[h][g] q_g,
// score_h = sum_G q'_h[G] . k_G.  So a query row of head h becomes nkv * hd lanes, one block per KV head, and the attention
// kernels (whose option for such wide rows adds up the blocks' products) need no other head's scores.
//  * rotate_heads     every head of a buffer turned in place by sign * position * freq[i] (the heads' weighted sums of
//                     rotated values turned back by the query's position).
//
// Norms, angles (a 32-bit product of position and frequency; the frequencies are rounded once from 64-bit on the host),
// sines and cosines are 32-bit.  A block a token; cosines and sines are computed once a token and shared by its heads.
// (Mixed queries of a few tokens: several blocks a token, each for some of its heads.)
#include "common.cuh"

namespace {

struct Rows {
    const float* p;
    int S;
    long long s_stride;
    long long ld;
};

__device__ __forceinline__ float rows_at(const Rows& in, long long t, int c) {
    float v = 0.f;
    const float* p = in.p + t * in.ld + c;
    for (int s = 0; s < in.S; ++s) v += p[(long long)s * in.s_stride];
    return v;
}

struct StoreArgs {
    Rows qkv;               // [T][nh hd + nkv hd (+ nkv vd)]
    const float* q_gain;    // [nh hd] or null: no norm over the whole projection
    const float* k_gain;    // [nkv hd]
    float eps;
    const int* positions;
    const float* freq;      // [rot / 2]
    const float* vfreq;     // [vrot / 2] or null: values are stored as they are
    const int* slot_map;    // token -> page * page_size + offset, -1: stored nowhere
    void* q_out;            // [T][nh hd]
    void* pages;            // a page: [nkv][page_size][hd] keys, then [nkv][page_size][vd] values
    long long page_stride;
    int page_size, num_pages;
    int nh, nkv, hd, vd, rot, vrot;
    int interleaved;        // pairing of the rotated lanes
    int v_from_k;           // values are the key lanes as projected (before norm and rotation); vd == hd
    int* status;
    const float* bias;      // [nh hd + nkv hd (+ nkv vd)] or null
    int unit_v;             // every value head divided by its root mean square (eps inside the root)
    const float* talk;      // [nh][nh] or null: queries mixed across heads, q_out is [T][nh][nkv * hd]
    int vec;                // rows, partial sums and bias lie on 16-byte words
    int talk_off;           // where the mixing matrix lies in shared memory (floats)
    float* gate_out;        // [T][n_gates] or null: sigmoids of the columns behind the projection's
    int n_gates;            // nh, or nh * vd: one per lane of the heads' results
    float* v_keep;          // [T][nkv vd] or null: receives the values as projected
    const float* v_first;   // [T][nkv vd] or null: an earlier layer's values of the same tokens
    const float* v_share;   // how much of them is mixed in (one number)
};

// lanes (a, b) of pair k of a head whose first `dims` lanes turn; b < 0: lane a passes unchanged
__device__ __forceinline__ void pair_lanes(int k, int dims, int interleaved, int& a, int& b) {
    const int half = dims >> 1;
    if (k < half) {
        a = interleaved ? 2 * k : k;
        b = interleaved ? 2 * k + 1 : k + half;
    } else {
        a = dims + (k - half);
        b = -1;
    }
}

template <typename TC> __device__ __forceinline__ void store_pair(TC* p, float x, float y);
template <> __device__ __forceinline__ void store_pair<float>(float* p, float x, float y) { *reinterpret_cast<float2*>(p) = make_float2(x, y); }
template <> __device__ __forceinline__ void store_pair<__nv_bfloat16>(__nv_bfloat16* p, float x, float y) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(x, y);
}

template <typename TC>
__global__ void qkv_rope_store_kernel(StoreArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int nq = a.nh * a.hd, nk = a.nkv * a.hd, nv = a.v_from_k ? 0 : a.nkv * a.vd;
    const int n = nq + nk + nv;
    float* row = sm;                    // [n]
    float* cs = sm + n;                 // [rot]: cosines, then sines
    float* vcs = cs + a.rot;            // [vrot]
    float* vscale = vcs + a.vrot;       // [nkv] with unit values
    const int nh4 = (a.nh + 3) & ~3;
    float* talk = sm + a.talk_off;      // [nh][nh4] with mixed queries, transposed: weights of head g's queries in all heads' scores
    const float pos = (float)a.positions[t];
    const int half = a.rot >> 1, vhalf = a.vrot >> 1;
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * a.freq[i], &cs[half + i], &cs[i]);
    if (a.vfreq != nullptr)
        for (int i = threadIdx.x; i < vhalf; i += blockDim.x) sincosf(pos * a.vfreq[i], &vcs[vhalf + i], &vcs[i]);
    float sq = 0.f, sk = 0.f;
    const float share = a.v_first != nullptr ? *a.v_share : 0.f;
    // what becomes of lane c of the values on its way into the row
    auto value_lane = [&](int c, float v) {
        const size_t at = (size_t)t * nv + (c - nq - nk);
        if (a.v_keep != nullptr) a.v_keep[at] = v;
        return a.v_first != nullptr ? fmaf(share, a.v_first[at] - v, v) : v;
    };
    const bool mixes = a.v_keep != nullptr || a.v_first != nullptr;
    const bool first = blockIdx.y == 0;     // (a token's further blocks only mix queries)
    const int n_mine = first ? n : nq;
    int from = 0;
    if (a.vec) {        // 16-byte words, as far as whole ones go
        from = n_mine & ~3;
        for (int c = 4 * threadIdx.x; c < from; c += 4 * blockDim.x) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            const float* p = a.qkv.p + (long long)t * a.qkv.ld + c;
#pragma unroll 4
            for (int s = 0; s < a.qkv.S; ++s) {
                const float4 w = *reinterpret_cast<const float4*>(p + (long long)s * a.qkv.s_stride);
                v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
            }
            if (a.bias != nullptr) {
                const float4 b = *reinterpret_cast<const float4*>(a.bias + c);
                v.x += b.x; v.y += b.y; v.z += b.z; v.w += b.w;
            }
            if (mixes && c + 3 >= nq + nk) {
                float* f = reinterpret_cast<float*>(&v);
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (c + k >= nq + nk) f[k] = value_lane(c + k, f[k]);
            }
            *reinterpret_cast<float4*>(row + c) = v;
            if (a.q_gain != nullptr) {
                const float f[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    if (c + k < nq) sq = fmaf(f[k], f[k], sq);
                    else if (c + k < nq + nk) sk = fmaf(f[k], f[k], sk);
                }
            }
        }
    }
    for (int c = from + threadIdx.x; c < n_mine; c += blockDim.x) {
        float v = rows_at(a.qkv, t, c);
        if (a.bias != nullptr) v += a.bias[c];
        if (mixes && c >= nq + nk) v = value_lane(c, v);
        row[c] = v;
        if (c < nq) sq = fmaf(v, v, sq);
        else if (c < nq + nk) sk = fmaf(v, v, sk);
    }
    if (a.gate_out != nullptr && first) {
        int h0 = 0;
        if (a.vec && (n & 3) == 0 && (a.n_gates & 3) == 0) {
            h0 = a.n_gates;
            for (int h = 4 * threadIdx.x; h < h0; h += 4 * blockDim.x) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                const float* p = a.qkv.p + (long long)t * a.qkv.ld + n + h;
#pragma unroll 4
                for (int s = 0; s < a.qkv.S; ++s) {
                    const float4 w = *reinterpret_cast<const float4*>(p + (long long)s * a.qkv.s_stride);
                    v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
                }
                *reinterpret_cast<float4*>(a.gate_out + (size_t)t * a.n_gates + h) =
                    make_float4(1.f / (1.f + expf(-v.x)), 1.f / (1.f + expf(-v.y)), 1.f / (1.f + expf(-v.z)), 1.f / (1.f + expf(-v.w)));
            }
        }
        for (int h = h0 + threadIdx.x; h < a.n_gates; h += blockDim.x)
            a.gate_out[(size_t)t * a.n_gates + h] = 1.f / (1.f + expf(-rows_at(a.qkv, t, n + h)));
    }
    if (a.talk != nullptr)
        for (int i = threadIdx.x; i < a.nh * nh4; i += blockDim.x) {
            const int g = i / nh4, h = i % nh4;
            talk[i] = h < a.nh ? a.talk[h * a.nh + g] : 0.f;
        }
    float rq = 1.f, rk = 1.f;
    if (a.q_gain != nullptr) {
        sq = block_sum(sq, red);
        sk = block_sum(sk, red);
        rq = 1.0f / sqrtf(sq / (float)nq + a.eps);
        rk = 1.0f / sqrtf(sk / (float)nk + a.eps);
    } else __syncthreads();
    if (a.unit_v && first) {
        // a warp a value head; the factors are read behind the next barrier
        const int lane = threadIdx.x & 31;
        for (int g = threadIdx.x >> 5; g < a.nkv; g += blockDim.x >> 5) {
            const float* v = row + (a.v_from_k ? nq + g * a.hd : nq + nk + g * a.vd);
            float ss = 0.f;
            for (int c = lane; c < a.vd; c += 32) ss = fmaf(v[c], v[c], ss);
            ss = warp_sum(ss);
            if (lane == 0) vscale[g] = 1.0f / sqrtf(ss / (float)a.vd + a.eps);
        }
    }
    const int per_q = half + (a.hd - 2 * half);
    if (a.talk != nullptr) {
        // the queries turned in place, then mixed: 4 heads and two neighbouring lanes of one KV head's block a thread
        for (int i = threadIdx.x; i < a.nh * half; i += blockDim.x) {
            const int k = i % half;
            float* p = row + (i / half) * a.hd;
            int la, lb;
            pair_lanes(k, a.rot, a.interleaved, la, lb);
            const float x = p[la], y = p[lb], c = cs[k], s = cs[half + k];
            p[la] = x * c - y * s;
            p[lb] = y * c + x * s;
        }
        __syncthreads();
        const int gs = a.nh / a.nkv, wide = a.nkv * a.hd, pairs = (a.hd + 1) / 2;
        const bool even = (a.hd & 1) == 0;
        TC* wq = (TC*)a.q_out + (size_t)t * a.nh * wide;
        const int hb = ((a.nh + 3) / 4 - (int)blockIdx.y + (int)gridDim.y - 1) / (int)gridDim.y;     // this block's fours of heads
        for (int i = threadIdx.x; i < hb * a.nkv * pairs; i += blockDim.x) {
            const int d = 2 * (i % pairs), G = (i / pairs) % a.nkv, h0 = 4 * ((i / (pairs * a.nkv)) * (int)gridDim.y + (int)blockIdx.y);
            const bool two = even || d + 1 < a.hd;
            const float* src = row + (size_t)G * gs * a.hd + d;
            float acc[4][2];
#pragma unroll
            for (int m = 0; m < 4; ++m) acc[m][0] = acc[m][1] = 0.f;
            for (int g = 0; g < gs; ++g) {
                float x, y;
                if (even) {
                    const float2 xy = *reinterpret_cast<const float2*>(src + g * a.hd);
                    x = xy.x;
                    y = xy.y;
                } else {
                    x = src[g * a.hd];
                    y = two ? src[g * a.hd + 1] : 0.f;
                }
                const float4 w4 = *reinterpret_cast<const float4*>(talk + (G * gs + g) * nh4 + h0);
                const float w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
                for (int m = 0; m < 4; ++m) {
                    acc[m][0] = fmaf(w[m], x, acc[m][0]);
                    acc[m][1] = fmaf(w[m], y, acc[m][1]);
                }
            }
#pragma unroll
            for (int m = 0; m < 4; ++m) {
                if (h0 + m < a.nh) {
                    TC* dst = wq + (size_t)(h0 + m) * wide + G * a.hd + d;
                    if (even) store_pair<TC>(dst, acc[m][0], acc[m][1]);
                    else {
                        dst[0] = from_f32<TC>(acc[m][0]);
                        if (two) dst[1] = from_f32<TC>(acc[m][1]);
                    }
                }
            }
        }
    } else if (a.unit_v) __syncthreads();
    // queries
    TC* q_out = (TC*)a.q_out + (size_t)t * nq;
    for (int i = threadIdx.x; a.talk == nullptr && i < a.nh * per_q; i += blockDim.x) {
        const int h = i / per_q, base = h * a.hd;
        int la, lb;
        pair_lanes(i % per_q, a.rot, a.interleaved, la, lb);
        const float x = row[base + la] * (a.q_gain ? rq * a.q_gain[base + la] : 1.f);
        if (lb < 0) q_out[base + la] = from_f32<TC>(x);
        else {
            const float y = row[base + lb] * (a.q_gain ? rq * a.q_gain[base + lb] : 1.f);
            const float c = cs[i % per_q], s = cs[half + i % per_q];
            q_out[base + la] = from_f32<TC>(x * c - y * s);
            q_out[base + lb] = from_f32<TC>(y * c + x * s);
        }
    }
    const int slot = a.slot_map[t];
    if (slot < 0 || !first) return;
    const int page = slot / a.page_size, off = slot % a.page_size;
    if (page >= a.num_pages) {
        if (threadIdx.x == 0) atomicOr(a.status, VCB_STATUS_BAD_PAGE);
        return;
    }
    TC* kp = (TC*)a.pages + (size_t)page * a.page_stride;
    TC* vp = kp + (size_t)a.nkv * a.page_size * a.hd;
    // keys
    for (int i = threadIdx.x; i < a.nkv * per_q; i += blockDim.x) {
        const int g = i / per_q, base = nq + g * a.hd;
        TC* dst = kp + ((size_t)g * a.page_size + off) * a.hd;
        int la, lb;
        pair_lanes(i % per_q, a.rot, a.interleaved, la, lb);
        const float x = row[base + la] * (a.k_gain ? rk * a.k_gain[g * a.hd + la] : 1.f);
        if (lb < 0) dst[la] = from_f32<TC>(x);
        else {
            const float y = row[base + lb] * (a.k_gain ? rk * a.k_gain[g * a.hd + lb] : 1.f);
            const float c = cs[i % per_q], s = cs[half + i % per_q];
            dst[la] = from_f32<TC>(x * c - y * s);
            dst[lb] = from_f32<TC>(y * c + x * s);
        }
    }
    // values
    const int vr = a.vfreq != nullptr ? a.vrot : 0;
    const int per_v = (vr >> 1) + (a.vd - 2 * (vr >> 1));
    for (int i = threadIdx.x; i < a.nkv * per_v; i += blockDim.x) {
        const int g = i / per_v, base = a.v_from_k ? nq + g * a.hd : nq + nk + g * a.vd;
        TC* dst = vp + ((size_t)g * a.page_size + off) * a.vd;
        int la, lb;
        pair_lanes(i % per_v, vr, a.interleaved, la, lb);
        const float vs = a.unit_v ? vscale[g] : 1.f;
        const float x = row[base + la] * vs;
        if (lb < 0) dst[la] = from_f32<TC>(x);
        else {
            const float y = row[base + lb] * vs;
            const float c = vcs[i % per_v], s = vcs[vhalf + i % per_v];
            dst[la] = from_f32<TC>(x * c - y * s);
            dst[lb] = from_f32<TC>(y * c + x * s);
        }
    }
}

template <typename TC>
__global__ void rotate_heads_kernel(TC* x, const int* __restrict__ positions, const float* __restrict__ freq, float sign, int H,
                                    int width, int dims, int interleaved) {
    extern __shared__ float cs[];       // [dims]
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, half = dims >> 1;
    const float pos = sign * (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * freq[i], &cs[half + i], &cs[i]);
    __syncthreads();
    TC* row = x + (size_t)t * H * width;
    for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
        const int h = i / half, k = i % half;
        int la, lb;
        pair_lanes(k, dims, interleaved, la, lb);
        TC* p = row + (size_t)h * width;
        const float u = to_f32(p[la]), v = to_f32(p[lb]);
        p[la] = from_f32<TC>(u * cs[k] - v * cs[half + k]);
        p[lb] = from_f32<TC>(v * cs[k] + u * cs[half + k]);
    }
}

}  // namespace

// qkv [S][T][ld] 32-bit sums; q_out [T][nh hd] and the pages of `dtype`; vfreq null: values stored unturned.
// bias, talk (q_out then [T][nh][nkv hd]), gate_out with n_gates, v_keep, v_first with v_share (or null each) and unit_v: the
// options of StoreArgs.
VCB_API int vcb_qkv_rope_store(const float* qkv, int S, long long s_stride, long long ld, const float* q_gain, const float* k_gain,
                               float eps, const int* positions, const float* freq, const float* vfreq, const int* slot_map,
                               void* q_out, void* pages, long long page_stride, int page_size, int num_pages, int nh, int nkv,
                               int hd, int vd, int rot, int vrot, int interleaved, int v_from_k, int T, int dtype, int* status,
                               const float* bias, int unit_v, const float* talk, float* gate_out, int n_gates, float* v_keep,
                               const float* v_first, const float* v_share, cudaStream_t stream) {
    if (T == 0) return 0;
    VCB_CHECK_ARG(nh > 0 && nkv > 0 && hd > 0 && vd > 0, "qkv_rope_store: bad sizes %d %d %d %d", nh, nkv, hd, vd);
    VCB_CHECK_ARG(rot >= 0 && rot <= hd && rot % 2 == 0, "qkv_rope_store: %d turning lanes of %d", rot, hd);
    VCB_CHECK_ARG(vfreq == nullptr || (vrot >= 0 && vrot <= vd && vrot % 2 == 0), "qkv_rope_store: %d turning value lanes of %d", vrot, vd);
    VCB_CHECK_ARG(!v_from_k || vd == hd, "qkv_rope_store: keys that double as values have their size (%d, not %d)", hd, vd);
    VCB_CHECK_ARG((q_gain == nullptr) == (k_gain == nullptr), "qkv_rope_store: one gain without the other");
    VCB_CHECK_ARG(rot == 0 || freq != nullptr, "qkv_rope_store: no frequencies");
    StoreArgs a{Rows{qkv, S < 1 ? 1 : S, s_stride, ld}, q_gain, k_gain, eps, positions, freq, vfreq, slot_map, q_out, pages, page_stride,
                page_size, num_pages, nh, nkv, hd, vd, rot, vfreq ? vrot : 0, interleaved, v_from_k, status, bias, unit_v, talk, 0, 0, gate_out, n_gates, v_keep, v_first, v_share};
    VCB_CHECK_ARG(gate_out == nullptr || n_gates == nh || n_gates == nh * vd, "qkv_rope_store: %d gates for %d heads of %d lanes", n_gates, nh, vd);
    VCB_CHECK_ARG((v_keep == nullptr && v_first == nullptr) || !v_from_k, "qkv_rope_store: keys that double as values are not mixed");
    VCB_CHECK_ARG(v_first == nullptr || v_share != nullptr, "qkv_rope_store: values to mix in without a share");
    a.vec = (uintptr_t)qkv % 16 == 0 && (uintptr_t)bias % 16 == 0 && ld % 4 == 0 && (S <= 1 || s_stride % 4 == 0) && (uintptr_t)gate_out % 16 == 0;
    const int nh4 = (nh + 3) & ~3;
    a.talk_off = ((nh * hd + nkv * hd + (v_from_k ? 0 : nkv * vd) + rot + (vfreq ? vrot : 0) + (unit_v ? nkv : 0)) + 3) & ~3;
    const size_t smem = talk ? (size_t)(a.talk_off + nh * nh4) * sizeof(float) : (size_t)(nh * hd + nkv * hd + (v_from_k ? 0 : nkv * vd) + rot + (vfreq ? vrot : 0)
                                 + (unit_v ? nkv : 0)) * sizeof(float);
    VCB_CHECK_ARG(talk == nullptr || nh % nkv == 0, "qkv_rope_store: %d heads mixed over %d KV heads", nh, nkv);
    VCB_CHECK_ARG(talk == nullptr || q_gain == nullptr, "qkv_rope_store: mixed queries come without a norm over the whole projection");
    VCB_CHECK_ARG(smem <= 200 * 1024, "qkv_rope_store: a token's %zu bytes are more than the kernel's shared memory holds", smem);
    auto kern = dtype == VCB_F32 ? qkv_rope_store_kernel<float> : qkv_rope_store_kernel<__nv_bfloat16>;
    if (smem + 1024 > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
        vcb_set_error("qkv_rope_store: %zu bytes of shared memory refused", smem);
        return -2;
    }
    // few tokens with queries to mix: a token's heads are dealt to several blocks
    const int fours = (nh + 3) / 4;
    const int split = talk == nullptr || T > 64 ? 1 : (fours < 8 ? fours : 8);
    launch_pdl(kern, dim3(T, split), dim3(256), smem, stream, a);
    VCB_CHECK_LAUNCH("qkv_rope_store");
    return 0;
}

// x [T][H][width] of `dtype`, in place: the first `dims` lanes of every head turn by sign * position * freq[i].
VCB_API int vcb_rotate_heads(void* x, int dtype, const int* positions, const float* freq, float sign, int T, int H, int width,
                             int dims, int interleaved, cudaStream_t stream) {
    if (T == 0 || H == 0 || dims == 0) return 0;
    VCB_CHECK_ARG(dims > 0 && dims <= width && dims % 2 == 0, "rotate_heads: %d turning lanes of %d", dims, width);
    const size_t smem = (size_t)dims * sizeof(float);
    const int threads = H * dims / 2 >= 256 ? 256 : 128;
    if (dtype == VCB_F32)
        launch_pdl(rotate_heads_kernel<float>, dim3(T), dim3(threads), smem, stream, (float*)x, positions, freq, sign, H, width, dims, interleaved);
    else
        launch_pdl(rotate_heads_kernel<__nv_bfloat16>, dim3(T), dim3(threads), smem, stream, (__nv_bfloat16*)x, positions, freq, sign, H, width,
                   dims, interleaved);
    VCB_CHECK_LAUNCH("rotate_heads");
    return 0;
}
