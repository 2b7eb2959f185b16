// Attention of grouped heads over the chunk pool on tensor cores (bf16, mma.sync): decode items of the planner's work
// list, and portions of prompts for head sizes the tcgen05 kernel (ca_attn_span.cu) does not take.
//
// A CTA works for one key/value head on a block of query rows against a list of chunks.  The rows are the query heads
// of the group for consecutive tokens: row r is head r % group of token r / group, so the K/V that are staged once serve
// every query head that reads them.
//   decode    block = an item of the work list (one sequence's private chunks, or a run that several share);
//             emits one partial (running max, sum, un-normalised O) per row, combined by rows_merge_kernel
//   portions  block = up to 64 rows of consecutive tokens of a span over the span's chunks, each row up to its own
//             position; emits finished rows
// Four warps; up to 16 rows the warps split every tile's 64 tokens four ways, up to 32 rows two ways, else each warp has
// its own 16 rows.  K and V arrive by 16-byte asynchronous copies in a ring of stages, laid out as 128-byte lines
// whose granules are XOR-ed with the token number (conflict-free ldmatrix).  Softmax is online, in fp32 and log2 units; the
// weights enter the second product as a sum of two bf16 numbers, which keeps 16 bits of them.
#include <algorithm>

#include "ca_kernels.h"
#include "ca_plan.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int R_THREADS = 128, R_TILE = 64;
constexpr float R_NEG_BIG = -1.0e30f;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool valid) {
    const int n = valid ? 16 : 0;  // 0: the destination is filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// a pair of weights as the bf16 pairs hi + lo
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
// byte offset of granule g of token t in a staged tile: panels of [64 tokens][128 bytes]
__device__ __forceinline__ uint32_t staged(int t, int g) { return (g >> 3) * (R_TILE * 128) + t * 128 + (((g & 7) ^ (t & 7)) << 4); }

// Scores, softmax and O += P V of one warp: 16 rows against 16 * NS tokens of the staged tile from token tb.
template <int DK, int DV, int NS>
__device__ __forceinline__ void warp_tile(uint32_t k_tile, uint32_t v_tile, int tb, int first, const uint32_t (&qf)[DK / 16][4],
                                          const int (&limit)[2], float scale_log2, float (&m)[2], float (&l)[2],
                                          float (&o)[DV / 8][4], int lane) {
    float s[2 * NS][4];
#pragma unroll
    for (int i = 0; i < 2 * NS; i++)
#pragma unroll
        for (int k = 0; k < 4; k++) s[i][k] = 0.f;
    const int mat = lane >> 3, r = lane & 7;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ks++)
#pragma unroll
        for (int sl = 0; sl < NS; sl++) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4(b0, b1, b2, b3, k_tile + staged(tb + 16 * sl + (mat >> 1) * 8 + r, 2 * ks + (mat & 1)));
            mma_bf16(s[2 * sl], qf[ks], b0, b1);
            mma_bf16(s[2 * sl + 1], qf[ks], b2, b3);
        }
    const int col = first + tb + (lane & 3) * 2;  // token of s[i][0] is col + 8 i
    float mx[2] = {R_NEG_BIG, R_NEG_BIG};
#pragma unroll
    for (int i = 0; i < 2 * NS; i++)
#pragma unroll
        for (int k = 0; k < 4; k++) {
            s[i][k] = col + 8 * i + (k & 1) < limit[k >> 1] ? s[i][k] * scale_log2 : -INFINITY;
            mx[k >> 1] = fmaxf(mx[k >> 1], s[i][k]);
        }
    float alpha[2], sum[2] = {0.f, 0.f};
#pragma unroll
    for (int h = 0; h < 2; h++) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        const float mn = fmaxf(m[h], mx[h]);
        alpha[h] = fast_exp2(m[h] - mn);
        m[h] = mn;
    }
#pragma unroll
    for (int i = 0; i < 2 * NS; i++)
#pragma unroll
        for (int k = 0; k < 4; k++) {
            s[i][k] = fast_exp2(s[i][k] - m[k >> 1]);
            sum[k >> 1] += s[i][k];
        }
    l[0] = l[0] * alpha[0] + sum[0];  // this lane's columns only: summed over the quad at the end
    l[1] = l[1] * alpha[1] + sum[1];
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
        for (int i = 0; i < DV / 8; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) o[i][k] *= alpha[k >> 1];
    }
#pragma unroll
    for (int sl = 0; sl < NS; sl++) {
        uint32_t hi[4], lo[4];
        split_bf16(s[2 * sl][0], s[2 * sl][1], hi[0], lo[0]);
        split_bf16(s[2 * sl][2], s[2 * sl][3], hi[1], lo[1]);
        split_bf16(s[2 * sl + 1][0], s[2 * sl + 1][1], hi[2], lo[2]);
        split_bf16(s[2 * sl + 1][2], s[2 * sl + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int dt = 0; dt < DV / 16; dt++) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(b0, b1, b2, b3, v_tile + staged(tb + 16 * sl + (mat & 1) * 8 + r, 2 * dt + (mat >> 1)));
            mma_bf16(o[2 * dt], hi, b0, b1);
            mma_bf16(o[2 * dt], lo, b0, b1);
            mma_bf16(o[2 * dt + 1], hi, b2, b3);
            mma_bf16(o[2 * dt + 1], lo, b2, b3);
        }
    }
}

// BULK: chunks of 64 tokens whose tiles are exactly DK and DV wide are staged verbatim (the pool's layout is the staged one)
// by 1-D TMA bulk copies of one thread.
template <int DK, int DV, int STAGES, bool SPAN, bool BULK>
__global__ void __launch_bounds__(R_THREADS) rows_mma_kernel(const RowsParams p) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int K_BYTES = R_TILE * DK * 2, STAGE_BYTES = R_TILE * (DK + DV) * 2;
    const uint32_t sbase = smem_u32(smem);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int G = p.geo.n_heads, group = p.group, H = G * group, C = p.geo.chunk_size;

    // ---- the block of rows and its chunks
    int kvh, token0, n_rows, n_ctx, slot_base = 0, row_lo = 0;
    const int32_t* list;
    if (SPAN) {
        const int sub = blockIdx.x % p.subs;
        kvh = blockIdx.y;
        const int4 b = reinterpret_cast<const int4*>(p.blocks)[blockIdx.x / p.subs];
        token0 = b.y;
        n_rows = (b.z - b.y) * group;
        row_lo = sub * 64;
        if (row_lo >= n_rows) return;
        n_rows = min(64, n_rows - row_lo);
        list = p.path_chunks + p.path_off[b.x];
        n_ctx = p.positions[token0 + (row_lo + n_rows - 1) / group] + 1;
    } else {
        const int idx = (int)blockIdx.x / G;
        kvh = blockIdx.x % G;
        const int* it = reinterpret_cast<const int*>(p.items) + 16 * idx;
        const int n_tiles = it[0], flags = it[5], last = it[6];
        token0 = it[2];
        n_rows = it[3] * group;
        slot_base = it[4];
        list = it + 7;
        n_ctx = (n_tiles - 1) * C + min(C, last + ((flags & ITEM_FLAG_TAIL) ? p.delta_tokens : 0));
        row_lo = (int)blockIdx.y * 64;
        if (row_lo >= n_rows) return;
        n_rows = min(64, n_rows - row_lo);
    }
    const int splits = n_rows <= 16 ? 4 : (n_rows <= 32 ? 2 : 1);
    const int my_m = splits == 4 ? 0 : (splits == 2 ? (warp & 1) : warp);      // 16-row tile of this warp
    const int my_s = splits == 4 ? warp : (splits == 2 ? (warp >> 1) : 0);     // its share of the tokens
    const bool busy = my_m * 16 < n_rows;

    // ---- staging
    const int gpr = p.geo.gpr, v_gpr = p.geo.v_gpr;
    const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(p.pool);
    const int n_tiles = (n_ctx + R_TILE - 1) / R_TILE;
    const uint32_t bars = sbase + STAGES * STAGE_BYTES;  // BULK: one barrier per stage
    if (BULK) {
        if (tid == 0) {
            for (int i = 0; i < STAGES; i++) mbar_init(bars + 8 * i, 1);
            asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        }
        __syncthreads();
    }
    auto copy_tile = [&](int j) {  // one thread
        const uint32_t dst = sbase + (j % STAGES) * STAGE_BYTES, bar = bars + 8 * (j % STAGES);
        int chunk = __ldg(list + j);
        if (chunk < 0 || chunk >= p.max_chunks) {
            atomicCAS(p.status, STATUS_OK, STATUS_BAD_WORK_LIST);
            chunk = 0;
        }
        const uint8_t* src = static_cast<const uint8_t*>(p.pool) + ((size_t)chunk * G + kvh) * (size_t)STAGE_BYTES;
        const uint32_t lines = min(R_TILE, n_ctx - j * R_TILE);
        mbar_arrive_expect_tx(bar, lines * (DK + DV) * 2);
        if (lines == R_TILE) {
            bulk_copy_g2s(dst, src, STAGE_BYTES, bar);
        } else {
#pragma unroll
            for (int pn = 0; pn < (DK + DV) / 64; pn++) bulk_copy_g2s(dst + pn * (R_TILE * 128), src + pn * (R_TILE * 128), lines * 128, bar);
        }
    };
    // granules past the stored head size are zero in every stage
    if (!BULK) for (int i = tid; i < STAGES * R_TILE * (DK + DV) / 8; i += R_THREADS) {
        const int st = i / (R_TILE * (DK + DV) / 8), q = i % (R_TILE * (DK + DV) / 8);
        const bool is_k = q < R_TILE * DK / 8;
        const int qq = is_k ? q : q - R_TILE * DK / 8, t = qq % R_TILE, g = qq / R_TILE;
        if (g >= (is_k ? gpr : v_gpr)) sts128_zero(sbase + st * STAGE_BYTES + (is_k ? 0 : K_BYTES) + staged(t, g));
    }
    const int g_sub = tid & 7;
    auto load_tile = [&](int j) {
        const uint32_t dst = sbase + (j % STAGES) * STAGE_BYTES;
#pragma unroll
        for (int i = 0; i < R_TILE / 16; i++) {
            const int t = (tid >> 3) + 16 * i, tok = j * R_TILE + t;
            const bool valid = tok < n_ctx;
            const int at = valid ? tok : 0, row = at % C;
            const __nv_bfloat16* kt = pool + tile_base_elems(p.geo, list[at / C], kvh, 0);
            const __nv_bfloat16* vt = kt + p.geo.tile_elems;
#pragma unroll
            for (int pn = 0; pn < DK / 64; pn++) {
                const int g = pn * 8 + g_sub;
                if (g < gpr) {
                    const int64_t off = p.geo.swz ? ((int64_t)pn * C + row) * 8 + (g_sub ^ (row & 7)) : (int64_t)row * gpr + g;
                    cp_async16(dst + staged(t, g), kt + off * 8, valid);
                }
            }
#pragma unroll
            for (int pn = 0; pn < DV / 64; pn++) {
                const int g = pn * 8 + g_sub;
                if (g < v_gpr) {
                    const int64_t off = p.geo.v_swz ? ((int64_t)pn * C + row) * 8 + (g_sub ^ (row & 7)) : (int64_t)row * v_gpr + g;
                    cp_async16(dst + K_BYTES + staged(t, g), vt + off * 8, valid);
                }
            }
        }
    };
#pragma unroll
    for (int j = 0; j < STAGES - 1; j++) {
        if (BULK) {
            if (tid == 0 && j < n_tiles) copy_tile(j);
        } else {
            if (j < n_tiles) load_tile(j);
            cp_async_commit();
        }
    }

    // ---- queries, straight into fragments
    uint32_t qf[DK / 16][4];
    int limit[2];
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int r = my_m * 16 + (lane >> 2) + 8 * h;
        const bool on = r < n_rows;
        const int rr = row_lo + (on ? r : 0), token = token0 + rr / group;
        limit[h] = on ? (SPAN ? p.positions[token] + 1 : n_ctx) : 0;
        const uint32_t* q = reinterpret_cast<const uint32_t*>(static_cast<const __nv_bfloat16*>(p.q) +
                                                              ((size_t)token * H + kvh * group + rr % group) * p.geo.d_head);
#pragma unroll
        for (int ks = 0; ks < DK / 16; ks++)
#pragma unroll
            for (int k = 0; k < 2; k++) {
                const int e = ks * 16 + k * 8 + (lane & 3) * 2;
                qf[ks][2 * k + h] = on && e < p.geo.d_head ? q[e / 2] : 0u;
            }
    }
    float o[DV / 8][4], m[2] = {R_NEG_BIG, R_NEG_BIG}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int i = 0; i < DV / 8; i++)
#pragma unroll
        for (int k = 0; k < 4; k++) o[i][k] = 0.f;

    for (int j = 0; j < n_tiles; j++) {
        if (BULK) {
            bool ok = mbar_wait_bounded(bars + 8 * (j % STAGES), (j / STAGES) & 1, p.wait_limit);
            const int lines = n_ctx - j * R_TILE;
            if (lines < R_TILE) {
                // the rows of V behind the stored ones meet weights of zero and only have to be finite
                const uint32_t v = sbase + (j % STAGES) * STAGE_BYTES + K_BYTES;
                for (int i = tid; i < (DV / 64) * (R_TILE - lines) * 8; i += R_THREADS) {
                    const int pn = i / ((R_TILE - lines) * 8), q = i % ((R_TILE - lines) * 8);
                    sts128_zero(v + pn * (R_TILE * 128) + lines * 128 + q * 16);
                }
            }
            if (!__syncthreads_and(ok)) {
                // record it, wait (again with the limit) for the copies in flight, and leave the rows unwritten
                if (tid == 0) {
                    atomicCAS(p.status, STATUS_OK, STATUS_FULL_WAIT_TIMEOUT);
                    for (int f = j; f < min(n_tiles, j + STAGES - 1); f++)
                        mbar_wait_bounded(bars + 8 * (f % STAGES), (f / STAGES) & 1, p.wait_limit);
                }
                return;
            }
            if (tid == 0 && j + STAGES - 1 < n_tiles) copy_tile(j + STAGES - 1);
        } else {
            cp_async_wait<STAGES - 2>();
            __syncthreads();
            if (j + STAGES - 1 < n_tiles) load_tile(j + STAGES - 1);
            cp_async_commit();
        }
        const uint32_t kt = sbase + (j % STAGES) * STAGE_BYTES, vt = kt + K_BYTES;
        if (!busy) continue;
        if (splits == 4) warp_tile<DK, DV, 1>(kt, vt, my_s * 16, j * R_TILE, qf, limit, p.scale_log2, m, l, o, lane);
        else if (splits == 2) warp_tile<DK, DV, 2>(kt, vt, my_s * 32, j * R_TILE, qf, limit, p.scale_log2, m, l, o, lane);
        else warp_tile<DK, DV, 4>(kt, vt, 0, j * R_TILE, qf, limit, p.scale_log2, m, l, o, lane);
    }
    cp_async_wait<0>();
    __syncthreads();

    // ---- rows leave through shared memory, where the token splits meet
    constexpr int PITCH = DV + 4;
    float* stage = reinterpret_cast<float*>(smem);                  // [4 warps][16 rows][PITCH]
    float2* ml = reinterpret_cast<float2*>(stage + 4 * 16 * PITCH); // [4 warps][16 rows]
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const int r = warp * 16 + (lane >> 2) + 8 * h;
        if ((lane & 3) == 0) ml[r] = make_float2(m[h], l[h]);
#pragma unroll
        for (int i = 0; i < DV / 8; i++)
            *reinterpret_cast<float2*>(stage + r * PITCH + 8 * i + (lane & 3) * 2) = make_float2(o[i][2 * h], o[i][2 * h + 1]);
    }
    __syncthreads();
    const int m_step = splits == 1 ? 0 : (splits == 2 ? 32 : 16);  // rows between the splits of one row
    constexpr int LANES = R_THREADS / 16;                          // threads that share a row
    for (int r = tid / LANES; r < n_rows; r += 16) {
        float M = R_NEG_BIG, L = 0.f, w[4];
        for (int s = 0; s < splits; s++) M = fmaxf(M, ml[r + s * m_step].x);
        if (SPAN && p.sink) M = fmaxf(M, 0.f);
#pragma unroll
        for (int s = 0; s < 4; s++) {
            w[s] = s < splits ? fast_exp2(ml[r + s * m_step].x - M) : 0.f;
            if (s < splits) L = fmaf(w[s], ml[r + s * m_step].y, L);
        }
        const int rr = row_lo + r, token = token0 + rr / group, head = kvh * group + rr % group;
        if (SPAN) {
            if (p.sink) L += fast_exp2(-M);
            const float inv = L > 0.f ? 1.f / L : 0.f;
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + ((size_t)token * H + head) * p.out_width;
            const float pos = (float)p.positions[token];
            for (int i = tid % LANES; 2 * i < p.out_width; i += LANES) {
                float a = 0.f, b = 0.f;
                for (int s = 0; s < splits; s++) {
                    const float2 x = *reinterpret_cast<const float2*>(stage + (r + s * m_step) * PITCH + 2 * i);
                    a = fmaf(w[s], x.x, a);
                    b = fmaf(w[s], x.y, b);
                }
                a *= inv;
                b *= inv;
                if (p.value_freq) {
                    float sn, cs;
                    fast_sincos(pos * p.value_freq[i], &sn, &cs);
                    const float t = a * cs + b * sn;
                    b = b * cs - a * sn;
                    a = t;
                }
                out[2 * i] = __float2bfloat16_rn(a);
                if (2 * i + 1 < p.out_width) out[2 * i + 1] = __float2bfloat16_rn(b);
            }
        } else {
            const size_t slot = (size_t)(slot_base + rr / group) * H + head;
            if (tid % LANES == 0) p.part_ml[slot] = make_float2(M, L);
            float* dst = p.part_o + slot * p.part_width;
            for (int i = tid % LANES; 2 * i < p.part_width; i += LANES) {
                float a = 0.f, b = 0.f;
                for (int s = 0; s < splits; s++) {
                    const float2 x = *reinterpret_cast<const float2*>(stage + (r + s * m_step) * PITCH + 2 * i);
                    a = fmaf(w[s], x.x, a);
                    b = fmaf(w[s], x.y, b);
                }
                *reinterpret_cast<float2*>(dst + 2 * i) = make_float2(a, b);
            }
        }
    }
}

// One warp per (row, query head): combine the row's partials, add the sink, turn the result back, store.
template <int K>  // pairs of value elements per lane
__global__ void __launch_bounds__(256) rows_merge_kernel(const RowsParams p) {
    const int H = p.geo.n_heads * p.group;
    const int pair = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (pair >= p.n_rows * H) return;
    const int row = pair / H, head = pair % H;
    const int b = p.merge_off[row], n = p.merge_off[row + 1] - b;
    float M = p.sink ? 0.f : R_NEG_BIG;
    for (int i = lane; i < n; i += 32) M = fmaxf(M, p.part_ml[(size_t)p.merge_slots[b + i] * H + head].x);
    M = warp_max(M);
    float acc[K][2], L = p.sink && lane == 0 ? fast_exp2(-M) : 0.f;  // pairs lane + 32 k
#pragma unroll
    for (int k = 0; k < K; k++) acc[k][0] = acc[k][1] = 0.f;
    const int pairs = p.part_width / 2;
    for (int i0 = 0; i0 < n; i0 += 32) {
        size_t slot = 0;
        float w = 0.f;
        if (i0 + lane < n) {
            slot = (size_t)p.merge_slots[b + i0 + lane] * H + head;
            const float2 ml = p.part_ml[slot];
            w = fast_exp2(ml.x - M);
            L = fmaf(w, ml.y, L);
        }
        const int m = min(32, n - i0);
        constexpr int AHEAD = 8;  // partial rows requested together
        for (int ib = 0; ib < m; ib += AHEAD) {
            float2 x[AHEAD][K];
#pragma unroll
            for (int i = 0; i < AHEAD; i++) {
                const float* src = p.part_o + __shfl_sync(0xffffffffu, (unsigned long long)slot, (ib + i) & 31) * p.part_width;
#pragma unroll
                for (int k = 0; k < K; k++) {
                    const int q = lane + 32 * k;
                    x[i][k] = ib + i < m && q < pairs ? *reinterpret_cast<const float2*>(src + 2 * q) : make_float2(0.f, 0.f);
                }
            }
#pragma unroll
            for (int i = 0; i < AHEAD; i++) {
                const float wi = __shfl_sync(0xffffffffu, w, (ib + i) & 31);
#pragma unroll
                for (int k = 0; k < K; k++) {
                    acc[k][0] = fmaf(wi, x[i][k].x, acc[k][0]);
                    acc[k][1] = fmaf(wi, x[i][k].y, acc[k][1]);
                }
            }
        }
    }
    L = warp_sum(L);
    const float inv = L > 0.f ? 1.f / L : 0.f;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (size_t)pair * p.out_width;
    const float pos = p.positions ? (float)p.positions[row] : 0.f;
#pragma unroll
    for (int k = 0; k < K; k++) {
        const int i = lane + 32 * k;
        if (2 * i >= p.out_width) break;
        float a = acc[k][0] * inv, c = acc[k][1] * inv;
        if (p.value_freq) {
            float sn, cs;
            fast_sincos(pos * p.value_freq[i], &sn, &cs);
            const float t = a * cs + c * sn;
            c = c * cs - a * sn;
            a = t;
        }
        out[2 * i] = __float2bfloat16_rn(a);
        if (2 * i + 1 < p.out_width) out[2 * i + 1] = __float2bfloat16_rn(c);
    }
}

template <int DK, int DV, int STAGES, bool BULK>
cudaError_t launch(const RowsParams& p, cudaStream_t stream) {
    constexpr int ring = STAGES * R_TILE * (DK + DV) * 2 + (BULK ? STAGES * 8 : 0), out = 4 * 16 * (DV + 4) * 4 + 64 * 8;
    constexpr int smem = ring > out ? ring : out;
    auto* span = rows_mma_kernel<DK, DV, STAGES, true, BULK>;
    auto* items = rows_mma_kernel<DK, DV, STAGES, false, BULK>;
    auto* k = p.blocks ? span : items;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    if (p.blocks) {
        k<<<dim3(p.n_blocks * p.subs, p.geo.n_heads), R_THREADS, smem, stream>>>(p);
    } else {
        // an item has up to ITEM_ROWS query rows except when one token's group alone has more
        k<<<dim3(p.n_items * p.geo.n_heads, p.subs), R_THREADS, smem, stream>>>(p);
        e = cudaGetLastError();
        if (e != cudaSuccess) return e;
        const int64_t pairs = (int64_t)p.n_rows * p.geo.n_heads * p.group;
        const unsigned grid = (unsigned)((pairs + 7) / 8);
        if (p.part_width <= 64) rows_merge_kernel<1><<<grid, 256, 0, stream>>>(p);
        else if (p.part_width <= 128) rows_merge_kernel<2><<<grid, 256, 0, stream>>>(p);
        else rows_merge_kernel<4><<<grid, 256, 0, stream>>>(p);
    }
    return cudaGetLastError();
}

}  // namespace

cudaError_t launch_attn_rows(const RowsParams& p, cudaStream_t stream) {
    const int dk = p.geo.d_head, dv = p.geo.d_value;
    if (dk > 256 || dv > 256) return cudaErrorInvalidValue;
    if (p.geo.chunk_size == R_TILE) {  // tiles as the staged layout has them
        if (dk == 64 && dv == 64) return launch<64, 64, 4, true>(p, stream);
        if (dk == 64 && dv == 128) return launch<64, 128, 4, true>(p, stream);
        if (dk == 128 && dv == 64) return launch<128, 64, 4, true>(p, stream);
        if (dk == 128 && dv == 128) return launch<128, 128, 3, true>(p, stream);
    }
    if (dk <= 64) {
        if (dv <= 64) return launch<64, 64, 4, false>(p, stream);
        if (dv <= 128) return launch<64, 128, 3, false>(p, stream);
    } else if (dk <= 128) {
        if (dv <= 64) return launch<128, 64, 3, false>(p, stream);
        if (dv <= 128) return launch<128, 128, 3, false>(p, stream);
    }
    return launch<256, 256, 2, false>(p, stream);
}

}  // namespace ca
