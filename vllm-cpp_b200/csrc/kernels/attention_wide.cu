// Single decoded tokens whose query rows are wide (queries mixed across heads: a row has one block of head_dim lanes per KV
// head, and its score with a key position is the sum of the blocks' products with all the heads' keys there, see
// rope_store.cu), bfloat16, head_dim 64 or 128, pages of 8, 16, 32 or 64 tokens.
//
// Where every head reads every KV head's keys, a block per KV head would fetch all keys once per KV head.  So one block is
// a token and a slice of its keys with ALL query heads: keys and values come in once.  Per tile of up to 128 keys:
//
//   S = sum over KV heads of Q_block . K^T   mma.sync m16n8k16, a warp 16 keys of all rows (16 rows a tile of heads), the
//                    sums stay in registers over the KV heads;
//   softmax          the scores meet in shared memory, a warp a row in turn: running maximum and sum in 32-bit,
//                    P = exp(s - m) rounded to bfloat16;
//   O += P . V       per KV head the rows of its own query heads (up to 16), a warp head_dim / 8 of its value lanes; O stays
//                    in registers over the tiles.
//
// Two more warps bring in the pages by TMA, a stage each in turn (issuing a stage's copies takes a warp longer than the
// products on it take the others; one box per page through the grouped view of the cache, as attention_mma.cu does):
// a stage is a tile's keys (or values) of one KV head, keys first; it is as long as the slice's keys need, so that a short
// slice has more of them on their way.  Slices leave (maximum, sum,
// unnormalised output) partials for vcb_attn_merge.
//
// BLOCKS: the KV heads are blocks of one shared row (attention over latent rows wider than a tile, see attention.cu): all
// rows meet the values of every block, and a head's result is its blocks side by side.  Every wait is bounded and reports through the status word.
#include "common.cuh"
#include "mbarrier.cuh"
#include "kv_tensor_map.h"

#include <cuda.h>
#include <math_constants.h>

namespace {

constexpr int BN = 128;         // most keys of a tile
constexpr int NW = 8;           // multiplying warps
constexpr int NT = NW * 32;
constexpr int LW = 2;           // loading warps
constexpr int ITEM_INTS = 6;    // entry, q0, nq, slice, nslices, decode index (as in attention_mma.cu)
constexpr int MAX_SLOTS = 32;

struct WideArgs {
    const __nv_bfloat16* q;     // [tokens][nh][nkv * HD]
    __nv_bfloat16* out;         // [tokens][nh][HD]
    const int* block_table;
    const int* table_row;
    int max_blocks;
    const int* q_start;
    const int* q_len;
    const int* ctx_len;
    const int* items;
    float* part_o;
    float* part_ml;
    int nh, nkv, page_size, num_pages, window, chunked;
    float scale;
    const float* out_gate;      // [tokens][query heads] or null: what the result of a (token, head) is multiplied by
    int gate_lanes;             // out_gate is laid out as the result, a factor per lane
    int one_row;                // pages hold keys only: the values are the key rows
    const float* sink;          // [query heads] or null: the score of a silent key without a value in every softmax
    int ring_bytes;             // of shared memory for the stages
    int* status;
};

__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// a tile of `rows` rows of HD lanes as HD/64 pieces of [rows][128 bytes], 16-byte chunks swizzled by the row
__device__ __forceinline__ int swz_rows(int rows, int r, int c) { return (c >> 3) * (rows * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4); }
// the layout the page copies leave: [groups of 8 keys][halves of head_dim][8 rows][128 bytes]
template <int HALVES> __device__ __forceinline__ int swz_kv(int key, int c) {
    return (key >> 3) * (HALVES * 1024) + (c >> 3) * 1024 + (key & 7) * 128 + (((c & 7) ^ (key & 7)) << 4);
}
__device__ __forceinline__ void tma_load_groups(uint32_t dst, const CUtensorMap* map, uint32_t bar, int group) {
    asm volatile(
        "cp.async.bulk.tensor.4d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%3, %3, %3, %4}], [%2];"
        ::"r"(dst), "l"(map), "r"(bar), "r"(0), "r"(group) : "memory");
}
__device__ __forceinline__ void warps_barrier() { asm volatile("bar.sync 1, %0;" ::"n"(NT) : "memory"); }
__device__ __forceinline__ int first_key(int pos, int W, int chunked) {
    if (W <= 0) return 0;
    return max(0, chunked ? pos - pos % W : pos - W + 1);
}

constexpr int S_LD = BN + 4;      // floats of a row of scores in shared memory (its weights then lie over their first half)

// bytes behind the ring: the query rows, scores, weights, per-row numbers, barriers
__host__ __device__ inline int tail_bytes(int hd, int mt, int nkv) {
    const int rows = 16 * mt;
    return nkv * rows * hd * 2 + rows * S_LD * 4 + 3 * rows * 4 + 2 * MAX_SLOTS * 8 + 16;
}

// MT tiles of 16 rows hold the query heads; up to NG KV heads
template <int HD, int MT, int NG, bool BLOCKS = false>
__global__ __launch_bounds__(NT + 32 * LW, 1) void attn_wide_kernel(const __grid_constant__ CUtensorMap kv_map, WideArgs a) {
    constexpr int ROWS = 16 * MT, CH = HD / 8, ROWB = HD * 2, HALVES = HD / 64;
    constexpr int NTV = HD / 64;        // n-tiles of 8 value lanes a warp owns
    constexpr int MTV = BLOCKS ? MT : 1;        // tiles of 16 rows that meet a KV head's values
    constexpr float LOG2E = 1.4426950408889634f;
    extern __shared__ __align__(1024) uint8_t smem[];
    uint8_t* q_s = smem + a.ring_bytes;
    float* s_s = reinterpret_cast<float*>(q_s + a.nkv * ROWS * ROWB);       // [ROWS][S_LD]
    float* al_s = s_s + ROWS * S_LD;                                        // [ROWS] rescale factors of the tile
    float* m_s = al_s + ROWS;                                               // [ROWS] at the end: maxima, sums
    float* l_s = m_s + ROWS;
    uint8_t* bar_s = reinterpret_cast<uint8_t*>(l_s + ROWS);
    auto full_bar = [&](int st) { return smem_u32(bar_s) + 8u * st; };
    auto empty_bar = [&](int st) { return smem_u32(bar_s) + 8u * (MAX_SLOTS + st); };
    volatile int* abort_flag = reinterpret_cast<volatile int*>(bar_s + 16 * MAX_SLOTS);

    pdl_trigger();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int* item = a.items + (size_t)blockIdx.x * ITEM_INTS;
    const int e = item[0], slice = item[3], nslices = item[4], dec_index = item[5];
    const int qlen = a.q_len[e], ctx = a.ctx_len[e];
    // query rows; those that a KV head's values belong to; results of a token
    const int nh = BLOCKS ? a.nh / a.nkv : a.nh, nkv = a.nkv, gs = BLOCKS ? nh : nh / nkv, n_out = a.nh;
    if (qlen <= 0 || ctx <= 0 || (smem_u32(smem) & 1023u)) {
        pdl_wait();
        if (qlen > 0 && ctx > 0) {
            if (tid == 0) atomicOr(a.status, VCB_STATUS_BAD_LAYOUT);
        } else if (nslices > 1) {
            // an empty entry: its slices still say "nothing here", so that the merge writes zeros
            for (int h = tid; h < n_out; h += blockDim.x) {
                const size_t prow = ((size_t)dec_index * n_out + h) * nslices + slice;
                a.part_ml[prow * 2] = -CUDART_INF_F;
                a.part_ml[prow * 2 + 1] = 0.f;
            }
        }
        return;
    }
    const int row0 = a.q_start[e], pos = ctx - 1;
    const int ps = a.page_size;
    const int lo = first_key(pos, a.window, a.chunked), hi = pos + 1;
    const int pb_lo = lo / ps, pb_hi = (hi + ps - 1) / ps;
    const int pps = (pb_hi - pb_lo + nslices - 1) / nslices;
    const int my_lo = pb_lo + slice * pps, my_hi = min(pb_hi, my_lo + pps);
    const int k_begin = max(lo, my_lo * ps), k_end = min(hi, my_hi * ps);
    const int t_first = my_lo * ps;         // tiles start on a page boundary: whole pages come in
    const int tile_keys = min(BN, max(1, my_hi - my_lo) * ps);        // whole pages
    const int n_tiles = k_end > k_begin ? (k_end - t_first + tile_keys - 1) / tile_keys : 0;
    const int per_tile = 2 * nkv, n_loads = n_tiles * per_tile;     // a tile: nkv stages of keys, then nkv of values
    const int stage_bytes = tile_keys * ROWB;
    const int slots = min(MAX_SLOTS, a.ring_bytes / stage_bytes);

    if (tid == 0) {
        for (int st = 0; st < slots; ++st) {
            mbar_init(full_bar(st), 1);
            mbar_init(empty_bar(st), NW);
        }
        *abort_flag = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    __syncthreads();

    if (warp >= NW) {
        // ---- loads: every LW-th stage, a lane a page of the tile ----
        const int me = warp - NW;
        const int* bt = a.block_table + (size_t)(a.table_row ? a.table_row[e] : e) * a.max_blocks;
        const int pages_per_tile = tile_keys / ps, groups_page = ps / 8, groups_kv = a.one_row ? 0 : nkv * groups_page;
        auto page_of = [&](int tile) {
            const int pb = my_lo + tile * pages_per_tile + lane;
            return (tile < n_tiles && lane < pages_per_tile && pb < my_hi) ? bt[pb] : -1;
        };
        int page = page_of(0), next_page = page_of(1), tile_now = 0;
        auto issue = [&](int load) {
            const int tile = load / per_tile, sub = load % per_tile, st = load % slots;
            bool ok = true;
            if (load >= slots) {
                if (lane == 0) ok = mbar_wait(empty_bar(st), ((load / slots) & 1) ^ 1u, abort_flag, a.status);
                if (!__shfl_sync(0xffffffffu, ok, 0)) return false;
            }
            while (tile_now < tile) {
                ++tile_now;
                page = next_page;
                next_page = page_of(tile_now + 1);
            }
            const int np = min(pages_per_tile, my_hi - (my_lo + tile * pages_per_tile));
            if (lane == 0) mbar_expect_tx(full_bar(st), (uint32_t)(np * ps * ROWB));
            __syncwarp();
            if (lane < np) {
                int p = page;
                if (p < 0 || p >= a.num_pages) {
                    atomicOr(a.status, VCB_STATUS_BAD_PAGE);
                    p = 0;      // keep the byte count whole; the status word reports the fault
                }
                const bool is_v = sub >= nkv;
                const int group = (p * (a.one_row ? 1 : 2) * nkv + (is_v ? sub - nkv : sub)) * groups_page + (is_v ? groups_kv : 0);
                tma_load_groups(smem_u32(smem + st * stage_bytes) + lane * ps * ROWB, &kv_map, full_bar(st), group);
            }
            return true;
        };
        // tiles whose pages hold only tokens of earlier steps are asked for before the wait
        int load = me;
        bool ok = true;
        while (ok && load < n_loads && load < slots &&
               min(my_hi, my_lo + (load / per_tile + 1) * pages_per_tile) * ps <= ctx - qlen)
        {
            ok = issue(load);
            load += LW;
        }
        pdl_wait();
        for (; ok && load < n_loads; load += LW) ok = issue(load);
        if (lane == 0 && *abort_flag) {     // let copies in flight land before the block goes away
            for (int i = load - LW; i >= 0 && i > load - LW - slots; i -= LW) {
                const long long c0 = clock64();
                while (!mbar_try(full_bar(i % slots), (i / slots) & 1) && clock64() - c0 < VCB_WAIT_CLOCKS) {}
            }
        }
        return;
    }

    pdl_wait();     // the queries and the newest key come from the kernel before this one
    const int q_ch = nkv * CH;
    for (int idx = tid; idx < ROWS * q_ch; idx += NT) {
        const int r = idx / q_ch, c = idx % q_ch;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n"
                     ::"r"(smem_u32(q_s + (c / CH) * (ROWS * ROWB) + swz_rows(ROWS, r, c % CH))),
                       "l"(a.q + ((size_t)row0 * nh + (r < nh ? r : 0)) * (nkv * HD) + c * 8), "r"(r < nh ? 16 : 0) : "memory");
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    float o[NG][MTV][NTV][4];
#pragma unroll
    for (int g = 0; g < NG; ++g)
#pragma unroll
        for (int m = 0; m < MTV; ++m)
#pragma unroll
            for (int n = 0; n < NTV; ++n) o[g][m][n][0] = o[g][m][n][1] = o[g][m][n][2] = o[g][m][n][3] = 0.f;
    float m_run[2 * MT], l_run[2 * MT];         // of rows warp, warp + 8, ... (every lane holds them)
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
        // (the silent key is the first slice's starting state)
        const bool sink = a.sink != nullptr && slice == 0 && warp + 8 * i < nh;
        m_run[i] = sink ? a.sink[warp + 8 * i] : -CUDART_INF_F;
        l_run[i] = sink ? 1.f : 0.f;
    }
    warps_barrier();

    // (a warp whose wait has run out goes on through the block's barriers without its products, so that none is left waiting)
    bool ok = true;
    const int mi = lane >> 3;
    for (int t = 0; t < n_tiles; ++t) {
        const int t0 = t_first + t * tile_keys, load0 = t * per_tile;
        // ---- S: this warp's 16 keys, all rows ----
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < 2; ++n) s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f;
        const int t_keys = min(tile_keys, k_end - t0);        // keys of this tile that count (from its start)
        for (int g = 0; g < nkv; ++g) {
            const int load = load0 + g, st = load % slots;
            if (ok) ok = mbar_wait(full_bar(st), (load / slots) & 1, abort_flag, a.status);
            if (!ok) break;
            const uint32_t kt = smem_u32(smem + st * stage_bytes), qb = smem_u32(q_s + g * (ROWS * ROWB));
            if (ok && warp * 16 < t_keys) {
                // (keys beyond the stage's are read off it -- whatever lies there, within the block's memory -- and masked)
#pragma unroll
                for (int ks = 0; ks < HD / 16; ++ks) {
                    uint32_t b[4];      // keys 0 .. 7 and 8 .. 15 of this warp's, 16 lanes each
                    ldmatrix_x4(b, kt + swz_kv<HALVES>(warp * 16 + (mi >> 1) * 8 + (lane & 7), ks * 2 + (mi & 1)));
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        uint32_t qf[4];
                        ldmatrix_x4(qf, qb + swz_rows(ROWS, m * 16 + (lane & 15), ks * 2 + (lane >> 4)));
                        mma_16816(s[m][0], qf, b[0], b[1]);
                        mma_16816(s[m][1], qf, b[2], b[3]);
                    }
                }
            }
            __syncwarp();
            if (lane == 0) mbar_arrive(empty_bar(st));
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const int c = warp * 16 + n * 8 + 2 * (lane & 3), key = t0 + c;
            const bool in0 = key >= k_begin && c < t_keys, in1 = key + 1 >= k_begin && c + 1 < t_keys;
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                float* dst = s_s + (m * 16 + (lane >> 2)) * S_LD + c;
                *reinterpret_cast<float2*>(dst) = make_float2(in0 ? s[m][n][0] * a.scale : -CUDART_INF_F, in1 ? s[m][n][1] * a.scale : -CUDART_INF_F);
                *reinterpret_cast<float2*>(dst + 8 * S_LD) = make_float2(in0 ? s[m][n][2] * a.scale : -CUDART_INF_F, in1 ? s[m][n][3] * a.scale : -CUDART_INF_F);
            }
        }
        warps_barrier();
        // ---- softmax: a warp a row in turn, four keys a lane ----
#pragma unroll
        for (int i = 0; i < 2 * MT; ++i) {
            const int r = warp + 8 * i;
            const float4 v = *reinterpret_cast<const float4*>(s_s + r * S_LD + 4 * lane);
            const float m_new = fmaxf(m_run[i], warp_max(fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w))));
            const float use = m_new == -CUDART_INF_F ? 0.f : m_new;
            const float alpha = exp2f((m_run[i] - use) * LOG2E);
            const float p0 = exp2f((v.x - use) * LOG2E), p1 = exp2f((v.y - use) * LOG2E), p2 = exp2f((v.z - use) * LOG2E), p3 = exp2f((v.w - use) * LOG2E);
            l_run[i] = l_run[i] * alpha + warp_sum((p0 + p1) + (p2 + p3));
            m_run[i] = m_new;
            const __nv_bfloat162 pa = __floats2bfloat162_rn(p0, p1), pc = __floats2bfloat162_rn(p2, p3);
            __syncwarp();       // (the row's scores have been read: its weights go over them)
            *reinterpret_cast<uint2*>(s_s + r * S_LD + 2 * lane) =
                make_uint2(*reinterpret_cast<const uint32_t*>(&pa), *reinterpret_cast<const uint32_t*>(&pc));
            if (lane == 0) al_s[r] = alpha;
        }
        warps_barrier();
        // ---- O += P V: per KV head its own query heads' rows, this warp's value lanes ----
#pragma unroll
        for (int g = 0; g < NG; ++g) {
            if (g < nkv && ok) {
                const int load = load0 + nkv + g, st = load % slots;
                ok = mbar_wait(full_bar(st), (load / slots) & 1, abort_flag, a.status);
                if (ok) {
                    uint8_t* vt = smem + st * stage_bytes;
                    const int k_rows = (t_keys + 31) & ~31;     // keys multiplied: those behind the last weigh nothing
                    const bool tail = t_keys < k_rows;
                    if (tail) {
                        // slots beyond the sequence and rows of pages that were not loaded: a zero weight times NaN is NaN
                        // (rows beyond the stage belong to the next one and are not touched: see below)
                        for (int idx = lane; idx < (min(k_rows, tile_keys) - t_keys) * NTV; idx += 32)
                            *reinterpret_cast<uint4*>(vt + swz_kv<HALVES>(t_keys + idx / NTV, warp * NTV + idx % NTV)) = make_uint4(0, 0, 0, 0);
                        __syncwarp();
                    }
                    const int r_first = BLOCKS ? 0 : g * gs;        // the first row that meets these values
                    const uint32_t vb = smem_u32(vt);
                    uint32_t pb[MTV];
#pragma unroll
                    for (int m = 0; m < MTV; ++m) {
                        const int ra = m * 16 + (lane >> 2);
                        const float al_a = al_s[r_first + min(ra, gs - 1)], al_b = al_s[r_first + min(ra + 8, gs - 1)];
#pragma unroll
                        for (int n = 0; n < NTV; ++n) {
                            o[g][m][n][0] *= al_a; o[g][m][n][1] *= al_a; o[g][m][n][2] *= al_b; o[g][m][n][3] *= al_b;
                        }
                        // (rows beyond the group's repeat its last: never read)
                        pb[m] = smem_u32(s_s + (r_first + min(m * 16 + (lane & 15), gs - 1)) * S_LD);
                    }
                    const int last_key = tile_keys - 8;     // (of the last group of eight in the stage)
                    for (int k0 = 0; k0 < k_rows; k0 += 32) {
                        uint32_t a0[MTV][4], a1[MTV][4], b[4];
#pragma unroll
                        for (int m = 0; m < MTV; ++m) {
                            ldmatrix_x4(a0[m], pb[m] + k0 * 2 + (lane >> 4) * 16);
                            ldmatrix_x4(a1[m], pb[m] + k0 * 2 + 32 + (lane >> 4) * 16);
                        }
                        // groups of eight keys beyond the stage: the last group once more (finite, and weighed by zero)
                        if constexpr (NTV == 2) {
                            ldmatrix_x4_trans(b, vb + swz_kv<HALVES>(min(k0 + (mi & 1) * 8, last_key) + (lane & 7), warp * 2 + (mi >> 1)));
#pragma unroll
                            for (int m = 0; m < MTV; ++m) {
                                mma_16816(o[g][m][0], a0[m], b[0], b[1]);
                                mma_16816(o[g][m][1], a0[m], b[2], b[3]);
                            }
                            ldmatrix_x4_trans(b, vb + swz_kv<HALVES>(min(k0 + 16 + (mi & 1) * 8, last_key) + (lane & 7), warp * 2 + (mi >> 1)));
#pragma unroll
                            for (int m = 0; m < MTV; ++m) {
                                mma_16816(o[g][m][0], a1[m], b[0], b[1]);
                                mma_16816(o[g][m][1], a1[m], b[2], b[3]);
                            }
                        } else {
                            ldmatrix_x4_trans(b, vb + swz_kv<HALVES>(min(k0 + mi * 8, last_key) + (lane & 7), warp));
#pragma unroll
                            for (int m = 0; m < MTV; ++m) {
                                mma_16816(o[g][m][0], a0[m], b[0], b[1]);
                                mma_16816(o[g][m][0], a1[m], b[2], b[3]);
                            }
                        }
                    }
                    if (tail) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      // the clearing stores above
                    __syncwarp();
                    if (lane == 0) mbar_arrive(empty_bar(st));
                }
            }
        }
        if (t + 1 < n_tiles) warps_barrier();       // (the next tile's scores go over these weights)
    }
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i)
        if (lane == 0) {
            m_s[warp + 8 * i] = m_run[i];
            l_s[warp + 8 * i] = l_run[i];
        }
    warps_barrier();
#pragma unroll
    for (int g = 0; g < NG; ++g) {
        if (g < nkv) {
#pragma unroll
            for (int i = 0; i < 2 * MTV; ++i) {
                const int m = i >> 1, half = i & 1;
                const int rg = m * 16 + (lane >> 2) + 8 * half, h = BLOCKS ? rg : g * gs + rg, oh = BLOCKS ? rg * nkv + g : h;
                if (rg < gs) {
                    float f = 1.f;
                    if (nslices == 1) {
                        f = l_s[h] > 0.f ? 1.f / l_s[h] : 0.f;
                        if (a.out_gate != nullptr && !a.gate_lanes) f *= a.out_gate[(size_t)row0 * nh + h];
                    }
                    const size_t prow = ((size_t)dec_index * n_out + oh) * nslices + slice;
#pragma unroll
                    for (int n = 0; n < NTV; ++n) {
                        const int d = (warp * NTV + n) * 8 + 2 * (lane & 3);
                        if (nslices == 1) {
                            const size_t at = ((size_t)row0 * n_out + oh) * HD + d;
                            const float2 gl = a.out_gate != nullptr && a.gate_lanes ? *reinterpret_cast<const float2*>(a.out_gate + at) : make_float2(1.f, 1.f);
                            *reinterpret_cast<__nv_bfloat162*>(a.out + at) =
                                __floats2bfloat162_rn(o[g][m][n][2 * half] * f * gl.x, o[g][m][n][2 * half + 1] * f * gl.y);
                        } else
                            *reinterpret_cast<float2*>(a.part_o + prow * HD + d) = make_float2(o[g][m][n][2 * half], o[g][m][n][2 * half + 1]);
                    }
                    if (nslices > 1 && warp == 0 && (lane & 3) == 0) {
                        a.part_ml[prow * 2] = m_s[h];
                        a.part_ml[prow * 2 + 1] = l_s[h];
                    }
                }
            }
        }
    }
}

constexpr int MAX_SMEM = 227 * 1024;

// shared memory that is left for the stages, in whole pieces of 1 KB (0: the query rows leave too little -- less than four
// stages of 64 keys)
int ring_bytes(int hd, int nh, int nkv) {
    const int mt = nh <= 16 ? 1 : (nh <= 32 ? 2 : 4);
    const int n = (MAX_SMEM - tail_bytes(hd, mt, nkv)) & ~1023;
    return n < 4 * 64 * hd * 2 ? 0 : n;
}

template <int HD, int MT, int NG, bool BLOCKS = false>
int launch(const CUtensorMap& map, const WideArgs& a, int n_items, cudaStream_t stream) {
    const size_t smem = (size_t)a.ring_bytes + tail_bytes(HD, MT, a.nkv);
    auto kern = attn_wide_kernel<HD, MT, NG, BLOCKS>;
    static size_t opted = 0;
    if (opted < smem) {
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) {
            vcb_set_error("attn_wide: %zu bytes of shared memory refused: %s", smem, cudaGetErrorString(e));
            return -2;
        }
        opted = smem;
    }
    launch_pdl(kern, dim3(n_items), dim3(NT + 32 * LW), smem, stream, map, a);
    VCB_CHECK_LAUNCH("attn_wide");
    return 0;
}

template <int HD, int MT>
int launch_heads(const CUtensorMap& map, const WideArgs& a, int n_items, cudaStream_t stream) {
    if (a.nkv <= 4) return launch<HD, MT, 4>(map, a, n_items, stream);
    if (a.nkv <= 8) return launch<HD, MT, 8>(map, a, n_items, stream);
    if constexpr (HD == 64) return launch<HD, MT, 16>(map, a, n_items, stream);
    return -1;
}

}  // namespace

// What the kernel takes for blocks of one shared row: up to 32 query heads, up to 8 blocks of 128 lanes.
VCB_API int vcb_attn_wide_blocks_supported(int dtype, int hd, int page_size, int query_heads, int blocks) {
    return dtype == VCB_BF16 && hd == 128 && (page_size == 8 || page_size == 16 || page_size == 32 || page_size == 64) &&
           query_heads >= 1 && query_heads <= (blocks <= 4 ? 32 : 16) && blocks >= 1 && blocks <= 8 && ring_bytes(hd, query_heads, blocks) > 0;
}

// What the kernel takes: up to 64 query heads, up to 16 of them (and 8 KV heads of 128 lanes, 16 of 64) a KV head.
VCB_API int vcb_attn_wide_supported(int dtype, int hd, int page_size, int nh, int nkv) {
    return dtype == VCB_BF16 && (hd == 64 || hd == 128) && (page_size == 8 || page_size == 16 || page_size == 32 || page_size == 64) &&
           nkv >= 1 && nh % nkv == 0 && nh <= 64 && nh / nkv <= 16 && nkv <= (hd == 64 ? 16 : 8) && ring_bytes(hd, nh, nkv) > 0;
}

// items: single tokens, [n_items][6] as vcb_attn_mma's; part_o [tokens][nh][slices][hd], part_ml [tokens][nh][slices][2] where
// items have several slices (merged by vcb_attn_merge, which then applies out_gate).
VCB_API int vcb_attn_wide(const void* q, void* out, const void* pages, long long page_stride, const int* block_table,
                          const int* table_row, int max_blocks, const int* q_start, const int* q_len, const int* ctx_len,
                          const int* items, int n_items, float* part_o, float* part_ml, int nh, int nkv, int hd, int page_size,
                          int num_pages, int window, int chunked, float scale, const float* out_gate, int gate_lanes, int one_row,
                          int blocks, const float* sink, int* status, cudaStream_t stream) {
    if (n_items == 0) return 0;
    VCB_CHECK_ARG(nh > 0 && nkv > 0 && nh % nkv == 0, "attn_wide: %d heads on %d KV heads", nh, nkv);
    const int rows = blocks ? nh / nkv : nh;
    VCB_CHECK_ARG(blocks ? vcb_attn_wide_blocks_supported(VCB_BF16, hd, page_size, rows, nkv) : vcb_attn_wide_supported(VCB_BF16, hd, page_size, nh, nkv), "attn_wide: %d heads on %d of %d lanes with pages of %d tokens are not supported", nh, nkv, hd, page_size);
    VCB_CHECK_ARG(window >= 0, "attn_wide: bad window %d", window);
    VCB_CHECK_ARG(((uintptr_t)pages % 16 == 0) && page_stride == (long long)(one_row ? 1 : 2) * nkv * page_size * hd,
                  "attn_wide: the pages of a layer must be contiguous and 16-byte aligned for TMA loads");
    VCB_CHECK_ARG((uintptr_t)q % 16 == 0, "attn_wide: q must be 16-byte aligned");
    CUtensorMap map;
    if (!vcb_kv_tensor_map(pages, (long long)num_pages * (one_row ? 1 : 2) * nkv * page_size, hd, page_size, &map, true)) return -3;
    WideArgs a{(const __nv_bfloat16*)q, (__nv_bfloat16*)out, block_table, table_row, max_blocks, q_start, q_len, ctx_len, items, part_o,
               part_ml, nh, nkv, page_size, num_pages, window, chunked, scale, out_gate, gate_lanes, one_row, sink, ring_bytes(hd, rows, nkv), status};
    if (blocks && nkv > 4) return launch<128, 1, 8, true>(map, a, n_items, stream);
    if (blocks) return rows <= 16 ? launch<128, 1, 4, true>(map, a, n_items, stream) : launch<128, 2, 4, true>(map, a, n_items, stream);
    if (hd == 64) return nh <= 16 ? launch_heads<64, 1>(map, a, n_items, stream) : nh <= 32 ? launch_heads<64, 2>(map, a, n_items, stream) : launch_heads<64, 4>(map, a, n_items, stream);
    return nh <= 16 ? launch_heads<128, 1>(map, a, n_items, stream) : nh <= 32 ? launch_heads<128, 2>(map, a, n_items, stream) : launch_heads<128, 4>(map, a, n_items, stream);
}
