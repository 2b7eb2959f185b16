// Attention of portions of prompts with keys and values expanded from a latent cache, on the Blackwell tensor path: per
// head, windowed and causal, tcgen05.mma (bf16) with accumulators in tensor memory, operands staged by TMA tensor copies.
//
// The expansion (one GEMM over the gathered rows of the step's windows) leaves a row-major matrix: per workspace row the
// unrotated keys of all heads, then their values; the rotated key part is a second, narrow matrix that the heads share.  A
// 64-element block of either is one TMA box with the 128-byte swizzle the tensor cores read, so a key tile is the boxes of
// its unrotated part followed by those of the rotated part, with no copy in between.  Boxes may reach into the next head:
// there the staged queries are zero, and columns of O past the value size are not stored.
//
// One CTA per (block of up to 256 consecutive tokens of a span, head).  Two groups of four warps own 128 query rows each and
// share every key and value tile of 64 tokens; a group takes part in the tiles its windows touch.
//   S = Q K^T   M = 128, N = 64; D in TMEM, two buffers per group, so that S of tile j + 1 is computed under softmax j
//   softmax     one thread per row (= TMEM lane), fp32, log2 units; only tiles on an edge of a window are masked; the
//               accumulator is rescaled when a row's maximum has grown by more than 8.  The weights go back over S as bf16
//               hi + lo parts, whose sum has 16 bits of the fp32 weight
//   O += P V    A = P from TMEM, B = the value tile (MN-major)
// and finishes its rows: the sink joins the denominator, bf16 rows leave through the group's query buffer.
// Warp roles: 0-3 and 4-7 the groups, 8 TMA producer, 9 TMEM and the MMA issue.
//
// Every wait is bounded: on expiry a status code is recorded, every role falls through to the common exit, and the TMEM
// columns are freed there.
#include <cuda.h>

#include "ca_kernels.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int E_ROWS = 128, E_GROUPS = 2, E_TOK = 64, E_THREADS = 320, E_MAX_STAGES = 4;
constexpr int E_COL_S = 128, E_COLS = 256;  // per group: O at column 0, S buffers from column 128
constexpr float E_NEG_BIG = -1.0e30f, E_RESCALE_STEP = 8.f, E_LOG2E = 1.4426950408889634f;

__host__ __device__ constexpr uint32_t idesc_bf16(int m, int n, bool b_mn_major) { return umma_idesc_f16(m, n, false, b_mn_major) | (1u << 7) | (1u << 10); }
__device__ __forceinline__ void report(int* status, int code) { atomicCAS(status, STATUS_OK, code); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float2 unpack_bf16(uint32_t v) { return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u)); }

// KP, VP: 64-element panels of a key and of a value
template <int KP, int VP> struct Sizes {
    static constexpr int Q_PANEL = E_ROWS * 128, Q_BYTES = KP * Q_PANEL;  // one group's queries
    static constexpr int K_PANEL = E_TOK * 128, K_BYTES = KP * K_PANEL, V_BYTES = VP * K_PANEL;
    static constexpr int LIMIT = 227 * 1024 - 512;
    static constexpr int ROOM = (LIMIT - E_GROUPS * Q_BYTES) / (K_BYTES + V_BYTES);
    static constexpr int STAGES = ROOM < E_MAX_STAGES ? ROOM : E_MAX_STAGES;
    static constexpr int BODY = E_GROUPS * Q_BYTES + STAGES * (K_BYTES + V_BYTES);
    static constexpr int NUM_BARS = 4 * STAGES + 6 * E_GROUPS;
    static constexpr int SMEM = BODY + NUM_BARS * 8 + 16;
    static_assert(STAGES >= 2 && SMEM <= 227 * 1024, "shared memory");
};

template <int KP, int VP>
__global__ void __launch_bounds__(E_THREADS, 1) latent_span_kernel(const LatentSpanParams p, const __grid_constant__ CUtensorMap kv_map,
                                                                   const __grid_constant__ CUtensorMap rot_map) {
    using Z = Sizes<KP, VP>;
    extern __shared__ __align__(1024) uint8_t smem[];
    const uint32_t sbase = smem_u32(smem);
    const uint32_t k_ring = sbase + E_GROUPS * Z::Q_BYTES, v_ring = k_ring + Z::STAGES * Z::K_BYTES;
    const uint32_t k_full = sbase + Z::BODY, k_empty = k_full + 8 * Z::STAGES;
    const uint32_t v_full = k_empty + 8 * Z::STAGES, v_empty = v_full + 8 * Z::STAGES;
    const uint32_t s_full = v_empty + 8 * Z::STAGES;        // [group][2]
    const uint32_t p_full = s_full + 16 * E_GROUPS;         // [group][2]
    const uint32_t o_done = p_full + 16 * E_GROUPS;         // [group]
    const uint32_t q_ready = o_done + 8 * E_GROUPS;         // [group]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Z::BODY + Z::NUM_BARS * 8);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = p.n_heads, head = blockIdx.x % H;
    const int4 blk = __ldg(reinterpret_cast<const int4*>(p.blocks) + blockIdx.x / H);
    const int token0 = blk.y, n_tok = blk.z - blk.y;
    const int pos0 = __ldg(p.positions + token0);           // the block's tokens are consecutive positions
    const int first = __ldg(p.first + blk.x), base = __ldg(p.base + blk.x);
    const int window = p.window > 0 ? p.window : 0x3fffffff;
    // tile j holds positions key0 + 64 j ..; group g takes tiles [lo, hi) of them
    const int key0 = max(first, pos0 - window + 1);
    const int row0 = base + key0 - first;
    auto group_rows = [&](int g) { return max(0, min(E_ROWS, n_tok - g * E_ROWS)); };
    auto tile_lo = [&](int g) { return max(0, pos0 + g * E_ROWS - window + 1 - key0) / E_TOK; };
    auto tile_hi = [&](int g) { return group_rows(g) > 0 ? (pos0 + g * E_ROWS + group_rows(g) - key0 + E_TOK - 1) / E_TOK : 0; };
    const int lo0 = tile_lo(0), hi0 = tile_hi(0);
    const int lo1 = group_rows(1) > 0 ? tile_lo(1) : 0, hi1 = tile_hi(1);
    const int n_tiles = max(hi0, hi1);

    if (threadIdx.x == 0) {
        for (int i = 0; i < Z::STAGES; i++) {
            mbar_init(k_full + 8 * i, 1);
            mbar_init(k_empty + 8 * i, 1);
            mbar_init(v_full + 8 * i, 1);
            mbar_init(v_empty + 8 * i, 1);
        }
        for (int g = 0; g < E_GROUPS; g++) {
            for (int b = 0; b < 2; b++) {
                mbar_init(s_full + 16 * g + 8 * b, 1);
                mbar_init(p_full + 16 * g + 8 * b, E_ROWS);
            }
            mbar_init(o_done + 8 * g, 1);
            mbar_init(q_ready + 8 * g, E_ROWS);
        }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 9) {  // the warp that allocates is the warp that frees
        tmem_alloc(smem_u32(tmem_slot), E_GROUPS * E_COLS);
        tmem_relinquish_alloc_permit();
    }
    tc_fence_before_thread_sync();
    __syncthreads();
    tc_fence_after_thread_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 8) {
        // ---- producer
        if (lane == 0) {
            int issued = 0;  // key and value tiles, alternating
            const int d_panels = (p.dim + 63) >> 6;
            for (int i = 0; i < 2 * n_tiles; i++) {
                const int j = i >> 1, slot = j % Z::STAGES, parity = ((j / Z::STAGES) & 1) ^ 1, row = row0 + j * E_TOK;
                const bool key = (i & 1) == 0;
                if (!mbar_wait_bounded((key ? k_empty : v_empty) + 8 * slot, parity, p.wait_limit)) {
                    report(p.status, STATUS_EMPTY_WAIT_TIMEOUT);
                    break;
                }
                const uint32_t bar = (key ? k_full : v_full) + 8 * slot;
                mbar_arrive_expect_tx(bar, key ? Z::K_BYTES : Z::V_BYTES);
                if (key) {
                    const uint32_t dst = k_ring + slot * Z::K_BYTES;
#pragma unroll
                    for (int pn = 0; pn < KP; pn++) {
                        if (pn < d_panels) tma_load_2d(dst + pn * Z::K_PANEL, &kv_map, head * p.dim + 64 * pn, row, bar);
                        else tma_load_2d(dst + pn * Z::K_PANEL, &rot_map, 64 * (pn - d_panels), row, bar);
                    }
                } else {
                    const uint32_t dst = v_ring + slot * Z::V_BYTES;
#pragma unroll
                    for (int pn = 0; pn < VP; pn++) tma_load_2d(dst + pn * Z::K_PANEL, &kv_map, H * p.dim + head * p.vdim + 64 * pn, row, bar);
                }
                issued++;
            }
            for (int f = issued > 2 * Z::STAGES ? issued - 2 * Z::STAGES : 0; f < issued; f++) {
                const int j = f >> 1;
                if (!mbar_wait_bounded(((f & 1) ? v_full : k_full) + 8 * (j % Z::STAGES), (j / Z::STAGES) & 1, p.wait_limit)) {
                    report(p.status, STATUS_DRAIN_TIMEOUT);
                    break;
                }
            }
        }
    } else if (warp == 9) {
        // ---- MMA issuer: one thread
        if (elect_one()) {
            bool live = true;
            constexpr uint32_t DESC_HI = umma_desc_sw128_hi(1024);
            constexpr uint32_t IDESC_QK = idesc_bf16(E_ROWS, E_TOK, false), IDESC_PV = idesc_bf16(E_ROWS, VP * 64, true);
            auto wait = [&](uint32_t bar, int parity) {
                if (live && !mbar_wait_bounded(bar, parity, p.wait_limit)) {
                    report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    live = false;
                }
            };
            auto takes = [&](int g, int j) { return g == 0 ? j >= lo0 && j < hi0 : j >= lo1 && j < hi1; };
            auto local = [&](int g, int j) { return j - (g == 0 ? lo0 : lo1); };
            auto issue_qk = [&](int j) {
                const int slot = j % Z::STAGES;
                wait(k_full + 8 * slot, (j / Z::STAGES) & 1);
                if (!live) return;
                tc_fence_after_thread_sync();
                const uint32_t b_lo = umma_desc_sw128_lo(k_ring + slot * Z::K_BYTES, 16);
#pragma unroll
                for (int g = 0; g < E_GROUPS; g++) {
                    if (!takes(g, j)) continue;
                    const int b = local(g, j) & 1;
                    const uint32_t d = tmem_base + g * E_COLS + E_COL_S + b * E_TOK;
                    const uint32_t q_lo = umma_desc_sw128_lo(sbase + g * Z::Q_BYTES, 16);
#pragma unroll
                    for (int ks = 0; ks < KP * 4; ks++) {
                        const uint64_t a = umma_desc_pack(q_lo + (((ks >> 2) * Z::Q_PANEL + (ks & 3) * 32) >> 4), DESC_HI);
                        const uint64_t bb = umma_desc_pack(b_lo + (((ks >> 2) * Z::K_PANEL + (ks & 3) * 32) >> 4), DESC_HI);
                        umma_ss_f16(d, a, bb, IDESC_QK, ks > 0 ? 1u : 0u);
                    }
                    umma_commit(s_full + 16 * g + 8 * b);
                }
                umma_commit(k_empty + 8 * slot);
            };
            wait(q_ready, 0);
            if (hi1 > 0) wait(q_ready + 8, 0);
            if (live) issue_qk(0);
            for (int j = 0; j < n_tiles && live; j++) {
                if (j + 1 < n_tiles) issue_qk(j + 1);
                const int slot = j % Z::STAGES;
                wait(v_full + 8 * slot, (j / Z::STAGES) & 1);
                const uint32_t v_lo = umma_desc_sw128_lo(v_ring + slot * Z::V_BYTES, Z::K_PANEL);
#pragma unroll
                for (int g = 0; g < E_GROUPS; g++) {
                    if (!takes(g, j)) continue;
                    const int i = local(g, j), b = i & 1;
                    wait(p_full + 16 * g + 8 * b, (i >> 1) & 1);
                    if (!live) break;
                    tc_fence_after_thread_sync();
                    const uint32_t d = tmem_base + g * E_COLS, a_tmem = d + E_COL_S + b * E_TOK;  // hi parts, then lo parts
#pragma unroll
                    for (int part = 0; part < 2; part++)
#pragma unroll
                        for (int kk = 0; kk < 4; kk++) {
                            const uint64_t bb = umma_desc_pack(v_lo + ((kk * 2048) >> 4), DESC_HI);
                            umma_ts_f16(d, a_tmem + part * 32 + kk * 8, bb, IDESC_PV, (i > 0 || kk > 0 || part > 0) ? 1u : 0u);
                        }
                    umma_commit(o_done + 8 * g);
                }
                if (live) umma_commit(v_empty + 8 * slot);
            }
        }
    } else {
        const int g = warp >> 2, r = threadIdx.x & (E_ROWS - 1), n_rows = group_rows(g);
        uint8_t* const q_smem = smem + g * Z::Q_BYTES;
        const uint32_t q_base = sbase + g * Z::Q_BYTES;
        if (n_rows > 0) {
            const int tok = token0 + g * E_ROWS, gpos = pos0 + g * E_ROWS;  // the group's first token and its position
            // ---- queries -> shared memory, K-major 128-byte-swizzled: the unrotated part as it comes, the rotated part
            // turned by the token's position, zeros elsewhere
            const int d_panels = (p.dim + 63) >> 6, width = p.dim + p.rot, half = p.rot / 2;
            const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q);
            auto line = [&](int row, int gran) { return q_base + (gran >> 3) * Z::Q_PANEL + row * 128 + (((gran & 7) ^ (row & 7)) << 4); };
            for (int i = r; i < E_ROWS * d_panels * 8; i += E_ROWS) {
                const int row = i / (d_panels * 8), gr = i % (d_panels * 8);
                uint4 v = make_uint4(0u, 0u, 0u, 0u);
                if (row < n_rows && 8 * gr < p.dim)
                    v = __ldg(reinterpret_cast<const uint4*>(q + ((size_t)(tok + row) * H + head) * width) + gr);
                sts128(line(row, gr), (int)v.x, (int)v.y, (int)v.z, (int)v.w);
            }
            const int rot_lines = (KP - d_panels) * 8;
            if (half % 8 == 0) {  // a unit is a granule of the first half and its partner in the second
                const int units = half / 8, tail = rot_lines - 2 * units;
                for (int i = r; i < E_ROWS * units; i += E_ROWS) {
                    const int row = i / units, u = i % units;
                    uint4 a = make_uint4(0u, 0u, 0u, 0u), b = a;
                    if (row < n_rows) {
                        const uint4* src = reinterpret_cast<const uint4*>(q + ((size_t)(tok + row) * H + head) * width + p.dim);
                        a = __ldg(src + u);
                        b = __ldg(src + units + u);
                        const float pos = (float)(gpos + row);
                        uint32_t* aw = reinterpret_cast<uint32_t*>(&a);
                        uint32_t* bw = reinterpret_cast<uint32_t*>(&b);
#pragma unroll
                        for (int k = 0; k < 4; k++) {
                            const float2 x = unpack_bf16(aw[k]), y = unpack_bf16(bw[k]);
                            float s0, c0, s1, c1;
                            fast_sincos(pos * __ldg(p.freq + 8 * u + 2 * k), &s0, &c0);
                            fast_sincos(pos * __ldg(p.freq + 8 * u + 2 * k + 1), &s1, &c1);
                            aw[k] = pack_bf16(x.x * c0 - y.x * s0, x.y * c1 - y.y * s1);
                            bw[k] = pack_bf16(y.x * c0 + x.x * s0, y.y * c1 + x.y * s1);
                        }
                    }
                    sts128(line(row, d_panels * 8 + u), (int)a.x, (int)a.y, (int)a.z, (int)a.w);
                    sts128(line(row, d_panels * 8 + units + u), (int)b.x, (int)b.y, (int)b.z, (int)b.w);
                }
                for (int i = r; i < E_ROWS * tail; i += E_ROWS) sts128_zero(line(i / tail, d_panels * 8 + 2 * units + i % tail));
            } else {
                for (int i = r; i < E_ROWS * rot_lines; i += E_ROWS) {
                    const int row = i / rot_lines, gr = i % rot_lines;
                    float x[8];
#pragma unroll
                    for (int k = 0; k < 8; k++) {
                        const int e = 8 * gr + k, pair = e < half ? e : e - half;
                        x[k] = 0.f;
                        if (row < n_rows && e < p.rot) {
                            const __nv_bfloat16* src = q + ((size_t)(tok + row) * H + head) * width + p.dim;
                            float sn, cs;
                            fast_sincos((float)(gpos + row) * __ldg(p.freq + pair), &sn, &cs);
                            const float a = __bfloat162float(src[pair]), b = __bfloat162float(src[pair + half]);
                            x[k] = e < half ? a * cs - b * sn : b * cs + a * sn;
                        }
                    }
                    sts128(line(row, d_panels * 8 + gr), (int)pack_bf16(x[0], x[1]), (int)pack_bf16(x[2], x[3]), (int)pack_bf16(x[4], x[5]), (int)pack_bf16(x[6], x[7]));
                }
            }
            fence_proxy_async();
            mbar_arrive(q_ready + 8 * g);

            // ---- softmax: thread r owns query row r of its group = TMEM lane r
            const bool active = r < n_rows;
            const int my_pos = gpos + r;
            const int lo = g == 0 ? lo0 : lo1, hi = g == 0 ? hi0 : hi1;
            const int seen_all = gpos + n_rows - window;  // from this position on, up to gpos, every row sees everything
            const float scale = p.scale_log2;
            const uint32_t lane_addr = tmem_base + g * E_COLS + ((uint32_t)((warp & 3) * 32) << 16);
            const uint32_t my_s = s_full + 16 * g, my_p = p_full + 16 * g, my_o = o_done + 8 * g;
            float m_used = E_NEG_BIG, l = 0.f;
            bool live = true;
            for (int i = 0; i < hi - lo && live; i++) {
                const int b = i & 1, k0 = key0 + (lo + i) * E_TOK;
                live = mbar_wait_bounded(my_s + 8 * b, (i >> 1) & 1, p.wait_limit);
                live = __all_sync(0xffffffffu, live);
                if (!live) {
                    if (lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    break;
                }
                tc_fence_after_thread_sync();
                uint32_t s0[32], s1[32];
                tmem_ld32(lane_addr + E_COL_S + b * E_TOK, s0);
                tmem_ld32(lane_addr + E_COL_S + b * E_TOK + 32, s1);
                tmem_wait_ld();
                if (k0 < seen_all || k0 + E_TOK - 1 > gpos) {
                    const int from = active ? my_pos - window + 1 - k0 : E_TOK, to = active ? my_pos - k0 : -1;
#pragma unroll
                    for (int c = 0; c < 32; c++) {
                        if (c < from || c > to) s0[c] = 0xff800000u;
                        if (32 + c < from || 32 + c > to) s1[c] = 0xff800000u;
                    }
                }
                float alpha = 1.f;
                bool rescale = false;
                {
                    float mx = fmaxf(__uint_as_float(s0[0]), __uint_as_float(s1[0]));
#pragma unroll
                    for (int c = 1; c < 32; c++) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[c]), __uint_as_float(s1[c])));
                    mx = fmaxf(mx * scale, E_NEG_BIG);
                    if (i == 0) {
                        m_used = mx;
                    } else if (mx > m_used + E_RESCALE_STEP) {
                        alpha = fast_exp2(m_used - mx);
                        m_used = mx;
                        l *= alpha;
                        rescale = true;
                    }
                }
                float sum = 0.f;
#pragma unroll
                for (int c = 0; c < 32; c++) {
                    s0[c] = __float_as_uint(fast_exp2(fmaf(__uint_as_float(s0[c]), scale, -m_used)));
                    s1[c] = __float_as_uint(fast_exp2(fmaf(__uint_as_float(s1[c]), scale, -m_used)));
                    sum += __uint_as_float(s0[c]) + __uint_as_float(s1[c]);
                }
                l += sum;
                uint32_t pk[32];
#pragma unroll
                for (int c = 0; c < 16; c++) {
                    pk[c] = pack_bf16(__uint_as_float(s0[2 * c]), __uint_as_float(s0[2 * c + 1]));
                    pk[16 + c] = pack_bf16(__uint_as_float(s1[2 * c]), __uint_as_float(s1[2 * c + 1]));
                }
                tmem_st32(lane_addr + E_COL_S + b * E_TOK, pk);
#pragma unroll
                for (int c = 0; c < 16; c++) {
                    const float2 a = unpack_bf16(pk[c]), d = unpack_bf16(pk[16 + c]);
                    pk[c] = pack_bf16(__uint_as_float(s0[2 * c]) - a.x, __uint_as_float(s0[2 * c + 1]) - a.y);
                    pk[16 + c] = pack_bf16(__uint_as_float(s1[2 * c]) - d.x, __uint_as_float(s1[2 * c + 1]) - d.y);
                }
                tmem_st32(lane_addr + E_COL_S + b * E_TOK + 32, pk);
                if (i > 0) {
                    // O += P V of tile i - 1 is complete (every thread follows o_done phase by phase)
                    live = mbar_wait_bounded(my_o, (i - 1) & 1, p.wait_limit);
                    live = __all_sync(0xffffffffu, live);
                    if (!live) {
                        if (lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                        break;
                    }
                }
                if (__any_sync(0xffffffffu, rescale)) {
                    tc_fence_after_thread_sync();
#pragma unroll
                    for (int c = 0; c < 2 * VP; c++) {
                        uint32_t o[32];
                        tmem_ld32(lane_addr + c * 32, o);
                        tmem_wait_ld();
#pragma unroll
                        for (int k = 0; k < 32; k++) o[k] = __float_as_uint(__uint_as_float(o[k]) * alpha);
                        tmem_st32(lane_addr + c * 32, o);
                    }
                }
                tmem_wait_st();
                tc_fence_before_thread_sync();
                mbar_arrive(my_p + 8 * b);
            }
            if (live) {
                live = mbar_wait_bounded(my_o, (hi - lo - 1) & 1, p.wait_limit);
                live = __all_sync(0xffffffffu, live);
                if (!live && lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
            }
            if (live) {
                tc_fence_after_thread_sync();
                // ---- epilogue: every MMA of the group has completed, so its query buffer is free; each warp its own 32 rows
                float inv;
                {
                    float total = l, M = m_used;
                    if (p.sink) {
                        const float sk = __ldg(p.sink + head) * E_LOG2E;
                        M = fmaxf(m_used, sk);
                        total = l * fast_exp2(m_used - M) + fast_exp2(sk - M);
                    }
                    inv = total > 0.f ? fast_exp2(m_used - M) / total : 0.f;
                }
#pragma unroll
                for (int c = 0; c < 2 * VP; c++) {
                    uint32_t o[32];
                    tmem_ld32(lane_addr + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int k = 0; k < 16; k++) o[k] = pack_bf16(__uint_as_float(o[2 * k]) * inv, __uint_as_float(o[2 * k + 1]) * inv);
#pragma unroll
                    for (int k = 0; k < 4; k++) sts128(line(r, 4 * c + k), (int)o[4 * k], (int)o[4 * k + 1], (int)o[4 * k + 2], (int)o[4 * k + 3]);
                }
                __syncwarp();
                const int wr = (warp & 3) * 32, rows_here = min(32, n_rows - wr), grans = p.vdim >> 3;
                __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
                for (int u = lane; u < rows_here * grans; u += 32) {
                    const int row = wr + u / grans, gr = u % grans;
                    const uint4 v = *reinterpret_cast<const uint4*>(q_smem + (line(row, gr) - q_base));
                    *(reinterpret_cast<uint4*>(out + ((size_t)(tok + row) * H + head) * p.vdim) + gr) = v;
                }
            }
        }
    }
    // ---- common exit: nobody touches TMEM after this barrier, then the allocating warp frees it
    tc_fence_before_thread_sync();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after_thread_sync();
        tmem_dealloc(tmem_base, E_GROUPS * E_COLS);
    }
}

using EncodeTiled = CUresult (*)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                 const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

EncodeTiled encoder() {
    static EncodeTiled fn = [] {
        void* f = nullptr;
        cudaDriverEntryPointQueryResult found;
        if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &f, cudaEnableDefault, &found) != cudaSuccess || found != cudaDriverEntryPointSuccess)
            f = nullptr;
        return reinterpret_cast<EncodeTiled>(f);
    }();
    return fn;
}

// row-major bf16 [rows, cols] with `stride` elements between rows, in boxes of 64 x 64
bool make_map(CUtensorMap* m, const void* data, int64_t rows, int64_t cols, int64_t stride) {
    const EncodeTiled encode = encoder();
    if (!encode) return false;
    const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)stride * 2};
    const cuuint32_t box[2] = {64, E_TOK}, step[2] = {1, 1};
    return encode(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(data), dims, strides, box, step, CU_TENSOR_MAP_INTERLEAVE_NONE,
                  CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int KP, int VP> cudaError_t launch(const LatentSpanParams& p, cudaStream_t stream) {
    using Z = Sizes<KP, VP>;
    CUtensorMap kv, rot;
    if (!make_map(&kv, p.kv, p.kv_rows, (int64_t)p.n_heads * (p.dim + p.vdim), p.kv_stride) ||
        !make_map(&rot, p.rot_keys, p.kv_rows, p.rot_stride, p.rot_stride))
        return cudaErrorInvalidValue;
    auto* k = latent_span_kernel<KP, VP>;
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, Z::SMEM);
    if (e != cudaSuccess) return e;
    k<<<p.n_blocks * p.n_heads, E_THREADS, Z::SMEM, stream>>>(p, kv, rot);
    return cudaGetLastError();
}

}  // namespace

bool latent_span_serves(int dim, int rot, int vdim) {
    return dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 && dim > 0 && dim <= 128 && rot <= 128 && vdim > 0 && vdim <= 128;
}
int latent_span_rot_panels(int rot) { return rot <= 64 ? 1 : 2; }

cudaError_t launch_latent_span(const LatentSpanParams& p, cudaStream_t stream) {
    const int kp = (p.dim + 63) / 64 + latent_span_rot_panels(p.rot), vp = (p.vdim + 63) / 64;
    if (!latent_span_serves(p.dim, p.rot, p.vdim) || p.rot_stride < 64 * latent_span_rot_panels(p.rot)) return cudaErrorInvalidValue;
    if (kp == 2) return vp == 1 ? launch<2, 1>(p, stream) : launch<2, 2>(p, stream);
    if (kp == 3) return vp == 1 ? launch<3, 1>(p, stream) : launch<3, 2>(p, stream);
    return vp == 1 ? launch<4, 1>(p, stream) : launch<4, 2>(p, stream);
}

}  // namespace ca
