// Attention whose keys and values are read out of one small latent vector per token.
//
// Per token the cache holds c (the normed latent, `kv_rank` lanes) and one rotated key part shared by all heads
// (`rot` lanes).  Head h's key is [W_uk[h] c | k_rot] and its value W_uv[h] c, so
//     q_h . k_h = (W_uk[h]^T q_h,plain) . c + q_h,rot . k_rot        and        sum_j w_j v_j = W_uv[h] (sum_j w_j c_j):
// with the queries carried into the latent space first, attention runs over the latent rows themselves as one shared
// KV head of kv_rank + rot key lanes whose values are the first kv_rank of them, and the heads' values are expanded
// afterwards.  The kernels here are the steps around that attention:
//
//  * latent_norm_rope_store   from the stacked down projections [q latent | kv latent | rotated key part] (32-bit sums):
//                             c_q = g_q n(q latent) to a buffer; c = g_kv n(kv latent) and the rotated key part to the
//                             token's cache row (key row [c | k_rot | zeros], and value row c unless the key rows double as
//                             values); optionally one gate per head from further columns (its sigmoid to a buffer)
//  * head_linear              out[t, h, :] = M[h] in[t, h, :] for every head's own small matrix (queries into the latent
//                             space, latent sums out to the heads' values)
//                             (long steps with bfloat16 matrices: on the tensor cores)
//  * rope_rows                the rotation alone, on a slice of every head of a 32-bit buffer (the queries' rotated part)
//
// Without a query latent (q_rank 0: queries straight from the input) the first of them has only the latter two to do.
// Rotation pairs lane i with lane i + dims / 2, or neighbouring lanes (`interleaved`); the angle is position * freq[i] in 32-bit, cos and sin times `gain`.
// Norms, angles and all sums are 32-bit.
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

struct LatentArgs {
    Rows u;                 // [T][q_rank + kv_rank + rot]
    const float* gq;        // [q_rank]
    const float* gkv;       // [kv_rank]
    float eps;
    const int* positions;
    const float* freq;      // [rot / 2]
    float gain;
    const int* slot_map;    // token -> page * page_size + offset, -1: stored nowhere
    void* cq_out;           // [T][q_rank]
    void* pages;
    long long page_stride;
    int page_size, num_pages;
    int q_rank, kv_rank, rot, T;
    int interleaved;        // lanes pair as neighbours
    int v_width;            // lanes of a value row: kv_rank, or more (the lanes behind the latent are zeros); 0: there are none
    int k_width;            // lanes of a key row: kv_rank + rot, or more (zeros)
    int k_block;            // a key row lies in pieces of this many lanes, all tokens' first pieces first (k_width: one piece)
    float* gate_out;        // [T][n_gates] or null: sigmoids of the columns behind the others
    int n_gates;
    int* status;
};

template <typename TC>
__global__ void latent_norm_rope_store_kernel(LatentArgs a) {
    extern __shared__ float row[];          // [q_rank + kv_rank + rot]
    __shared__ float red[33];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int nq = a.q_rank, nk = a.kv_rank, nr = a.rot, n = nq + nk + nr;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < n; c += blockDim.x) {
        const float v = rows_at(a.u, t, c);
        row[c] = v;
        if (c < nq) sq = fmaf(v, v, sq);
        else if (c < nq + nk) sk = fmaf(v, v, sk);
    }
    if (nq > 0) sq = block_sum(sq, red);
    sk = block_sum(sk, red);
    const float rq = nq > 0 ? rsqrtf(sq / (float)nq + a.eps) : 0.f, rk = rsqrtf(sk / (float)nk + a.eps);
    for (int h = threadIdx.x; h < a.n_gates; h += blockDim.x)
        a.gate_out[(size_t)t * a.n_gates + h] = 1.f / (1.f + expf(-rows_at(a.u, t, n + h)));
    TC* cq = (TC*)a.cq_out + (size_t)t * nq;
    for (int c = threadIdx.x; c < nq; c += blockDim.x) cq[c] = from_f32<TC>(row[c] * rq * a.gq[c]);
    const int slot = a.slot_map[t];
    if (slot < 0) return;
    const int page = slot / a.page_size, off = slot % a.page_size;
    if (page >= a.num_pages) {
        if (threadIdx.x == 0) atomicOr(a.status, VCB_STATUS_BAD_PAGE);
        return;
    }
    TC* base = (TC*)a.pages + (size_t)page * a.page_stride;
    auto key = [&](int c) -> TC& { return base[((size_t)(c / a.k_block) * a.page_size + off) * a.k_block + c % a.k_block]; };
    TC* vrow = base + (size_t)a.page_size * a.k_width + (size_t)off * a.v_width;
    for (int c = threadIdx.x; c < nk; c += blockDim.x) {
        const TC v = from_f32<TC>(row[nq + c] * rk * a.gkv[c]);
        key(c) = v;
        if (a.v_width > 0) vrow[c] = v;
    }
    for (int c = nk + nr + threadIdx.x; c < a.k_width; c += blockDim.x) key(c) = from_f32<TC>(0.f);
    for (int c = nk + threadIdx.x; c < a.v_width; c += blockDim.x) vrow[c] = from_f32<TC>(0.f);
    const int half = nr / 2;
    const float pos = (float)a.positions[t];
    const float* r = row + nq + nk;
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf(pos * a.freq[i], &sn, &cs);
        sn *= a.gain;
        cs *= a.gain;
        const int la = a.interleaved ? 2 * i : i, lb = a.interleaved ? 2 * i + 1 : i + half;
        const float x = r[la], y = r[lb];
        key(nk + la) = from_f32<TC>(x * cs - y * sn);
        key(nk + lb) = from_f32<TC>(y * cs + x * sn);
    }
    for (int i = 2 * half + threadIdx.x; i < nr; i += blockDim.x) key(nk + i) = from_f32<TC>(r[i]);
}

// One block: head h, a tile of TT tokens.  A warp an output lane: its lanes walk the inner dimension (coalesced reads of the
// matrix row), every token of the tile takes its sum from the same pass over that row.
constexpr int HL_TOKENS = 8;

struct HeadLinearArgs {
    const void* in;         // [S][T][ld_in]: 32-bit sums (in_dtype F32) or one buffer of the compute dtype
    int in_dtype;
    int S;
    long long s_stride, ld_in;
    int in_head_stride, in_off;     // head h reads lanes [h * in_head_stride + in_off, + n_in)
    const void* m;          // [H][n_out][n_in] in m_dtype
    int m_dtype;
    void* out;              // [T][ld_out] in out_dtype; head h writes lanes [h * out_head_stride + out_off, + n_out)
    int out_dtype;
    long long ld_out;
    int out_head_stride, out_off;
    int T, H, n_in, n_out;
};

__global__ void head_linear_kernel(HeadLinearArgs a) {
    extern __shared__ float x_s[];          // [HL_TOKENS][n_in]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, t0 = blockIdx.x * HL_TOKENS;
    const int nt = min(HL_TOKENS, a.T - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (int i = threadIdx.x; i < HL_TOKENS * a.n_in; i += blockDim.x) {
        const int tt = i / a.n_in, c = i % a.n_in;
        float v = 0.f;
        if (tt < nt) {
            const size_t at = (size_t)(t0 + tt) * a.ld_in + (size_t)h * a.in_head_stride + a.in_off + c;
            if (a.in_dtype == VCB_F32) {
                for (int s = 0; s < a.S; ++s) v += ((const float*)a.in)[at + (size_t)s * a.s_stride];
            } else {
                v = __bfloat162float(((const __nv_bfloat16*)a.in)[at]);
            }
        }
        x_s[i] = v;
    }
    __syncthreads();
    // (few tokens: a head's output lanes are dealt to several blocks)
    for (int j = blockIdx.z * nwarps + warp; j < a.n_out; j += gridDim.z * nwarps) {
        float acc[HL_TOKENS];
#pragma unroll
        for (int tt = 0; tt < HL_TOKENS; ++tt) acc[tt] = 0.f;
        const size_t mrow = ((size_t)h * a.n_out + j) * a.n_in;
        for (int c = lane; c < a.n_in; c += 32) {
            const float w = load_as_f32(a.m, a.m_dtype, mrow + c);
#pragma unroll
            for (int tt = 0; tt < HL_TOKENS; ++tt) acc[tt] = fmaf(w, x_s[tt * a.n_in + c], acc[tt]);
        }
#pragma unroll
        for (int tt = 0; tt < HL_TOKENS; ++tt) acc[tt] = warp_sum(acc[tt]);
        if (lane < nt) {
            float v = acc[0];
#pragma unroll
            for (int tt = 1; tt < HL_TOKENS; ++tt)
                if (lane == tt) v = acc[tt];
            store_from_f32(a.out, a.out_dtype, (size_t)(t0 + lane) * a.ld_out + (size_t)h * a.out_head_stride + a.out_off + j, v);
        }
    }
}

struct RopeArgs {
    Rows in;                // [T][...]: head h's slice starts at lane h * in_head_stride + in_off
    int in_head_stride, in_off;
    const int* positions;
    const float* freq;      // [dims / 2]
    float gain;
    void* out;
    int out_dtype;
    long long ld_out;
    int out_head_stride, out_off;
    int interleaved;
    int T, H, dims, width;  // `width` lanes of the slice are copied, the first `dims` of them rotated
    int pad;                // so many zero lanes go behind them
};

__global__ void rope_rows_kernel(RopeArgs a) {
    pdl_trigger();
    pdl_wait();
    const int half = a.dims / 2;
    const int per_head = half + (a.width - 2 * half) + a.pad;     // one thread a pair, one a lane that passes unchanged
    for (int t = blockIdx.y; t < a.T; t += gridDim.y) {
        const float pos = (float)a.positions[t];
        for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < a.H * per_head; i += gridDim.x * blockDim.x) {
            const int h = i / per_head, k = i % per_head;
            const int ib = h * a.in_head_stride + a.in_off;
            const size_t ob = (size_t)t * a.ld_out + (size_t)h * a.out_head_stride + a.out_off;
            if (k < half) {
                float sn, cs;
                sincosf(pos * a.freq[k], &sn, &cs);
                sn *= a.gain;
                cs *= a.gain;
                const int la = a.interleaved ? 2 * k : k, lb = a.interleaved ? 2 * k + 1 : k + half;
                const float x = rows_at(a.in, t, ib + la), y = rows_at(a.in, t, ib + lb);
                store_from_f32(a.out, a.out_dtype, ob + la, x * cs - y * sn);
                store_from_f32(a.out, a.out_dtype, ob + lb, y * cs + x * sn);
            } else {
                const int c = 2 * half + (k - half);
                store_from_f32(a.out, a.out_dtype, ob + c, c < a.width ? rows_at(a.in, t, ib + c) : 0.f);
            }
        }
    }
}

}  // namespace

// u [S][T][ld]: q_rank + kv_rank + rot columns.  cq_out [T][q_rank] and the pages in `dtype`.  A page is one flat row:
// [page_size][k_width] key rows (in pieces of k_block lanes, see LatentArgs), then [page_size][v_width] value rows (v_width >=
// kv_rank; the latent, then zeros: value rows as wide as key rows are what the tensor-core attention kernels read; 0: none,
// the key rows double as values).  gate_out [T][n_gates] (or null): sigmoids of n_gates columns behind the others.
VCB_API int vcb_latent_norm_rope_store(const float* u, int S, long long s_stride, long long ld, const float* gq, const float* gkv,
                                       float eps, const int* positions, const float* freq, float gain, const int* slot_map,
                                       void* cq_out, void* pages, long long page_stride, int page_size, int num_pages, int q_rank,
                                       int kv_rank, int rot, int interleaved, int k_width, int k_block, int v_width, float* gate_out, int n_gates,
                                       int T, int dtype, int* status, cudaStream_t stream) {
    if (T == 0) return 0;
    VCB_CHECK_ARG(q_rank >= 0 && kv_rank > 0 && rot >= 0, "latent_norm_rope_store: bad sizes %d %d %d", q_rank, kv_rank, rot);
    VCB_CHECK_ARG(k_width >= kv_rank + rot && k_block > 0 && k_width % k_block == 0, "latent_norm_rope_store: key rows of %d lanes in pieces of %d", k_width, k_block);
    VCB_CHECK_ARG(v_width == 0 || (v_width >= kv_rank && v_width <= k_width), "latent_norm_rope_store: value rows of %d lanes", v_width);
    VCB_CHECK_ARG(n_gates >= 0 && (n_gates == 0) == (gate_out == nullptr), "latent_norm_rope_store: %d gates without a buffer, or none with one", n_gates);
    LatentArgs a{Rows{u, S < 1 ? 1 : S, s_stride, ld}, gq, gkv, eps, positions, freq, gain, slot_map, cq_out, pages, page_stride,
                 page_size, num_pages, q_rank, kv_rank, rot, T, interleaved, v_width, k_width, k_block, gate_out, n_gates, status};
    const size_t smem = (size_t)(q_rank + kv_rank + rot) * sizeof(float);
    VCB_CHECK_ARG(smem <= 48 * 1024, "latent_norm_rope_store: %d lanes are more than the kernel's shared memory holds", q_rank + kv_rank + rot);
    if (dtype == VCB_F32) launch_pdl(latent_norm_rope_store_kernel<float>, dim3(T), dim3(256), smem, stream, a);
    else launch_pdl(latent_norm_rope_store_kernel<__nv_bfloat16>, dim3(T), dim3(256), smem, stream, a);
    VCB_CHECK_LAUNCH("latent_norm_rope_store");
    return 0;
}

// The same for a long step: one block is head h and HT_TOKENS tokens, a thread an output lane.  The thread walks its row of
// the matrix once (16 or 8 bytes at a time) and every token of the tile takes its sum from that pass, reading the token's
// inputs as 16-byte words that all threads share.  n_in is a multiple of four.
constexpr int HT_TOKENS = 32;

__global__ __launch_bounds__(128) void head_linear_tile_kernel(HeadLinearArgs a) {
    extern __shared__ __align__(16) float xt_s[];       // [HT_TOKENS][n_in]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, t0 = blockIdx.x * HT_TOKENS;
    const int nt = min(HT_TOKENS, a.T - t0);
    for (int i = threadIdx.x; i < HT_TOKENS * a.n_in; i += blockDim.x) {
        const int tt = i / a.n_in, c = i % a.n_in;
        float v = 0.f;
        if (tt < nt) {
            const size_t at = (size_t)(t0 + tt) * a.ld_in + (size_t)h * a.in_head_stride + a.in_off + c;
            if (a.in_dtype == VCB_F32) {
                for (int s = 0; s < a.S; ++s) v += ((const float*)a.in)[at + (size_t)s * a.s_stride];
            } else {
                v = __bfloat162float(((const __nv_bfloat16*)a.in)[at]);
            }
        }
        xt_s[i] = v;
    }
    __syncthreads();
    for (int j = threadIdx.x; j < a.n_out; j += blockDim.x) {
        float acc[HT_TOKENS];
#pragma unroll
        for (int tt = 0; tt < HT_TOKENS; ++tt) acc[tt] = 0.f;
        const size_t mrow = ((size_t)h * a.n_out + j) * a.n_in;
        for (int c = 0; c < a.n_in; c += 4) {
            float4 w;
            if (a.m_dtype == VCB_F32) {
                w = *reinterpret_cast<const float4*>((const float*)a.m + mrow + c);
            } else {
                const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)a.m + mrow + c);
                const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
                const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                w = make_float4(lo.x, lo.y, hi.x, hi.y);
            }
#pragma unroll
            for (int tt = 0; tt < HT_TOKENS; ++tt) {
                const float4 x = *reinterpret_cast<const float4*>(xt_s + tt * a.n_in + c);
                acc[tt] = fmaf(w.w, x.w, fmaf(w.z, x.z, fmaf(w.y, x.y, fmaf(w.x, x.x, acc[tt]))));
            }
        }
#pragma unroll
        for (int tt = 0; tt < HT_TOKENS; ++tt)
            if (tt < nt)
                store_from_f32(a.out, a.out_dtype, (size_t)(t0 + tt) * a.ld_out + (size_t)h * a.out_head_stride + a.out_off + j, acc[tt]);
    }
}

// The same on the tensor cores (mma.sync m16n8k16), for long steps with bfloat16 matrices: one block is head h and HM_TOKENS
// tokens, a warp 16 of them; the matrix comes in 64 rows at a time.  32-bit inputs go in as two bfloat16 parts, x = hi + lo
// (lo what rounding to hi leaves), two products into one 32-bit sum, so that they are not rounded on the way in.
constexpr int HM_TOKENS = 128, HM_OUT = 64, HM_THREADS = 256;

__device__ __forceinline__ uint32_t hm_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void hm_ldmatrix(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(hm_smem(p)));
}
__device__ __forceinline__ void hm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// lanes of a row in shared memory: whole steps of 16 and a pad that keeps neighbouring rows off the same banks
__host__ __device__ constexpr int hm_ld(int n_in) { return ((n_in + 15) & ~15) + 8; }

template <bool SPLIT>       // 32-bit inputs
__global__ __launch_bounds__(HM_THREADS) void head_linear_mma_kernel(HeadLinearArgs a) {
    extern __shared__ __align__(16) __nv_bfloat16 hm[];
    const int ld = hm_ld(a.n_in), K = ld - 8;
    __nv_bfloat16* x_hi = hm;                                               // [HM_TOKENS][ld]
    __nv_bfloat16* x_lo = x_hi + (SPLIT ? HM_TOKENS * ld : 0);              // [HM_TOKENS][ld]
    __nv_bfloat16* m_s = x_lo + HM_TOKENS * ld;                             // [HM_OUT][ld]
    pdl_trigger();
    pdl_wait();
    const int h = blockIdx.y, t0 = blockIdx.x * HM_TOKENS;
    const int nt = min(HM_TOKENS, a.T - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    // four lanes a thread, several loads in flight (16- or 8-byte words where rows and slices lie on them)
    const int quads = K / 4;
    const size_t elem = SPLIT ? 4 : 2;
    const bool words = ((a.n_in | a.in_head_stride | a.in_off | (int)(a.ld_in & 3) | (int)(a.s_stride & 3)) & 3) == 0 &&
                       (reinterpret_cast<uintptr_t>(a.in) & (4 * elem - 1)) == 0;
    auto fetch4 = [&](int idx) {
        const int tt = idx / quads, c = 4 * (idx % quads);
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
        if (idx >= HM_TOKENS * quads || tt >= nt || c >= a.n_in) return v;
        const size_t at = (size_t)(t0 + tt) * a.ld_in + (size_t)h * a.in_head_stride + a.in_off + c;
        float* f = reinterpret_cast<float*>(&v);
        if constexpr (SPLIT) {
            const float* p = (const float*)a.in + at;
            for (int s = 0; s < a.S; ++s, p += a.s_stride) {
                if (words) {
                    const float4 w = *reinterpret_cast<const float4*>(p);
                    v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
                } else {
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (c + k < a.n_in) f[k] += p[k];
                }
            }
        } else {
            const __nv_bfloat16* p = (const __nv_bfloat16*)a.in + at;
            if (words) {
                const uint2 raw = *reinterpret_cast<const uint2*>(p);
                const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
                const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
                v = make_float4(lo.x, lo.y, hi.x, hi.y);
            } else {
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    if (c + k < a.n_in) f[k] = __bfloat162float(p[k]);
            }
        }
        return v;
    };
    for (int i0 = threadIdx.x; i0 < HM_TOKENS * quads; i0 += 4 * HM_THREADS) {
        float4 v[4];
#pragma unroll
        for (int w = 0; w < 4; ++w) v[w] = fetch4(i0 + w * HM_THREADS);
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const int idx = i0 + w * HM_THREADS;
            if (idx < HM_TOKENS * quads) {
                const int at = (idx / quads) * ld + 4 * (idx % quads);
                const float f[4] = {v[w].x, v[w].y, v[w].z, v[w].w};
                __align__(8) __nv_bfloat16 hi[4], lo[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    hi[k] = __float2bfloat16_rn(f[k]);
                    lo[k] = __float2bfloat16_rn(f[k] - __bfloat162float(hi[k]));
                }
                *reinterpret_cast<uint2*>(x_hi + at) = *reinterpret_cast<const uint2*>(hi);
                if constexpr (SPLIT) *reinterpret_cast<uint2*>(x_lo + at) = *reinterpret_cast<const uint2*>(lo);
            }
        }
    }
    const __nv_bfloat16* m = (const __nv_bfloat16*)a.m + (size_t)h * a.n_out * a.n_in;
    const bool vec = (a.n_in & 7) == 0 && (reinterpret_cast<uintptr_t>(m) & 15) == 0;
    __nv_bfloat16* out = (__nv_bfloat16*)a.out + (size_t)h * a.out_head_stride + a.out_off;
    const bool pairs = ((a.out_head_stride | a.out_off | (int)a.ld_out) & 1) == 0 && (reinterpret_cast<uintptr_t>(a.out) & 3) == 0;
    for (int j0 = 0; j0 < a.n_out; j0 += HM_OUT) {
        if (vec) {
            const int ch = K / 8;
            for (int i = threadIdx.x; i < HM_OUT * ch; i += HM_THREADS) {
                const int j = i / ch, c = 8 * (i % ch);
                uint4 v = make_uint4(0, 0, 0, 0);
                if (j0 + j < a.n_out && c < a.n_in) v = *reinterpret_cast<const uint4*>(m + (size_t)(j0 + j) * a.n_in + c);
                *reinterpret_cast<uint4*>(m_s + j * ld + c) = v;
            }
        } else {
            for (int i = threadIdx.x; i < HM_OUT * K; i += HM_THREADS) {
                const int j = i / K, c = i % K;
                m_s[j * ld + c] = j0 + j < a.n_out && c < a.n_in ? m[(size_t)(j0 + j) * a.n_in + c] : __float2bfloat16_rn(0.f);
            }
        }
        __syncthreads();
        float acc[HM_OUT / 8][4];
#pragma unroll
        for (int n = 0; n < HM_OUT / 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
        const int xr = (warp * 16 + (lane & 15)) * ld + (lane >> 4) * 8;
        const int mr = ((lane >> 4) * 8 + (lane & 7)) * ld + ((lane >> 3) & 1) * 8;
        for (int k = 0; k < K; k += 16) {
            uint32_t xh[4], xl[4];
            hm_ldmatrix(xh, x_hi + xr + k);
            if constexpr (SPLIT) hm_ldmatrix(xl, x_lo + xr + k);
#pragma unroll
            for (int n = 0; n < HM_OUT / 16; ++n) {
                uint32_t b[4];
                hm_ldmatrix(b, m_s + n * 16 * ld + mr + k);
                hm_mma(acc[2 * n], xh, b[0], b[1]);
                hm_mma(acc[2 * n + 1], xh, b[2], b[3]);
                if constexpr (SPLIT) {
                    hm_mma(acc[2 * n], xl, b[0], b[1]);
                    hm_mma(acc[2 * n + 1], xl, b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int tt = warp * 16 + (lane >> 2) + 8 * half;
            if (tt < nt) {
                __nv_bfloat16* o = out + (size_t)(t0 + tt) * a.ld_out;
#pragma unroll
                for (int n = 0; n < HM_OUT / 8; ++n) {
                    const int j = j0 + n * 8 + 2 * (lane & 3);
                    const float u = acc[n][2 * half], v = acc[n][2 * half + 1];
                    if (pairs && j + 1 < a.n_out) *reinterpret_cast<__nv_bfloat162*>(o + j) = __floats2bfloat162_rn(u, v);
                    else {
                        if (j < a.n_out) o[j] = __float2bfloat16_rn(u);
                        if (j + 1 < a.n_out) o[j + 1] = __float2bfloat16_rn(v);
                    }
                }
            }
        }
        __syncthreads();
    }
}

VCB_API int vcb_head_linear(const void* in, int in_dtype, int S, long long s_stride, long long ld_in, int in_head_stride, int in_off,
                            const void* m, int m_dtype, void* out, int out_dtype, long long ld_out, int out_head_stride,
                            int out_off, int T, int H, int n_in, int n_out, cudaStream_t stream) {
    if (T == 0 || H == 0 || n_out == 0) return 0;
    VCB_CHECK_ARG(in_dtype == VCB_F32 || S <= 1, "head_linear: partial sums are 32-bit");
    const size_t smem = (size_t)HL_TOKENS * n_in * sizeof(float);
    VCB_CHECK_ARG(smem <= 48 * 1024, "head_linear: %d input lanes are more than the kernel's shared memory holds", n_in);
    VCB_CHECK_ARG(H <= 65535, "head_linear: %d heads", H);
    HeadLinearArgs a{in, in_dtype, S < 1 ? 1 : S, s_stride, ld_in, in_head_stride, in_off, m, m_dtype, out, out_dtype, ld_out,
                     out_head_stride, out_off, T, H, n_in, n_out};
    const bool split = in_dtype == VCB_F32;
    const size_t mma_smem = (size_t)(HM_TOKENS * (split ? 2 : 1) + HM_OUT) * hm_ld(n_in) * 2;
    if (T >= HM_TOKENS / 2 && m_dtype == VCB_BF16 && out_dtype == VCB_BF16 && mma_smem <= 200 * 1024) {
        auto kern = split ? head_linear_mma_kernel<true> : head_linear_mma_kernel<false>;
        if (mma_smem > 48 * 1024 && cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)mma_smem) != cudaSuccess) {
            vcb_set_error("head_linear: %zu bytes of shared memory refused", mma_smem);
            return -2;
        }
        launch_pdl(kern, dim3((T + HM_TOKENS - 1) / HM_TOKENS, H), dim3(HM_THREADS), mma_smem, stream, a);
        VCB_CHECK_LAUNCH("head_linear");
        return 0;
    }
    const size_t tile_smem = (size_t)HT_TOKENS * n_in * sizeof(float);
    if (T >= 2 * HT_TOKENS && (n_in & 3) == 0 && tile_smem <= 48 * 1024 && (reinterpret_cast<uintptr_t>(m) & 15) == 0) {
        launch_pdl(head_linear_tile_kernel, dim3((T + HT_TOKENS - 1) / HT_TOKENS, H), dim3(128), tile_smem, stream, a);
        VCB_CHECK_LAUNCH("head_linear");
        return 0;
    }
    const int token_blocks = (T + HL_TOKENS - 1) / HL_TOKENS;
    const int deal = token_blocks <= 4 ? (n_out + 31) / 32 : 1;
    launch_pdl(head_linear_kernel, dim3(token_blocks, H, deal < 64 ? deal : 64), dim3(256), smem, stream, a);
    VCB_CHECK_LAUNCH("head_linear");
    return 0;
}

VCB_API int vcb_rope_rows(const float* in, int S, long long s_stride, long long ld, int in_head_stride, int in_off,
                          const int* positions, const float* freq, float gain, void* out, int out_dtype, long long ld_out,
                          int out_head_stride, int out_off, int T, int H, int dims, int width, int pad, int interleaved, cudaStream_t stream) {
    if (T == 0 || H == 0 || width == 0) return 0;
    VCB_CHECK_ARG(pad >= 0 && dims >= 0 && dims <= width, "rope_rows: %d rotated lanes of %d", dims, width);
    RopeArgs a{Rows{in, S < 1 ? 1 : S, s_stride, ld}, in_head_stride, in_off, positions, freq, gain, out, out_dtype, ld_out,
               out_head_stride, out_off, interleaved, T, H, dims, width, pad};
    const int per_head = dims / 2 + (width - 2 * (dims / 2)) + pad;
    const dim3 grid((H * per_head + 127) / 128, T < 65535 ? T : 65535);
    launch_pdl(rope_rows_kernel, grid, dim3(128), 0, stream, a);
    VCB_CHECK_LAUNCH("rope_rows");
    return 0;
}
