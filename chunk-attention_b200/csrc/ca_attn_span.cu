// Causal attention of portions of prompts over the chunk pool on the Blackwell tensor path: tcgen05.mma (bf16) with
// accumulators in tensor memory, K/V chunks staged verbatim by 1-D TMA bulk copies.  For caches of 64-token chunks and
// head sizes of 64 or 128 elements, whose pool tiles are the tensor cores' own 128-byte-swizzled operand layout; other
// geometries take the mma.sync kernel (ca_attn_rows.cu).
//
// One CTA per (block of up to 128 query rows, key/value head).  The rows are the query heads of a group for consecutive
// tokens of one span (row r: head r % group of token r / group), and walk the span's chunks from position 0 to the last
// row's own position; only the tiles that reach past the first row's position are masked.
//   S = Q K^T      M = 128 rows, N = 64 tokens; A = the queries, staged once; B = a K tile; D in TMEM, two buffers, so that
//                  S of tile j + 1 is computed under the softmax of tile j
//   softmax        one thread per row (= TMEM lane), fp32, log2 units; the accumulator is rescaled only when a row's
//                  maximum has grown by more than 8.  The weights go back over S as bf16 hi + lo parts (SPLIT): their sum
//                  has 16 bits of the fp32 weight
//   O += P V       A = P from TMEM, B = the V tile (MN-major panels)
// and finishes its rows: sink, normalisation, the turn back of rotated values, bf16 store through shared memory.
// Warp roles: 0-3 softmax and epilogue, 4 TMA producer over a ring of four tile slots, 5 TMEM and the MMA issue.  Two
// CTAs share an SM, so one's softmax runs under the other's MMAs.
//
// Every wait is bounded: on expiry a status code is recorded, every role falls through to the common exit, and the TMEM
// columns are freed there.
#include "ca_kernels.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int A_ROWS = 128, A_TOK = 64, A_SLOTS = 4, A_THREADS = 192;
constexpr int A_TMEM_COLS = 256, A_COL_S = 128;
constexpr int A_NUM_BARS = 2 * A_SLOTS + 6;
constexpr float A_NEG_BIG = -1.0e30f, A_RESCALE_STEP = 8.f;

// tcgen05.mma.kind::f16 instruction descriptor with bf16 operands (formats 1 in both operand fields)
__host__ __device__ constexpr uint32_t idesc_bf16(int m, int n, bool b_mn_major) { return umma_idesc_f16(m, n, false, b_mn_major) | (1u << 7) | (1u << 10); }

__device__ __forceinline__ void report(int* status, int code) { atomicCAS(status, STATUS_OK, code); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}

template <int DK, int DV> struct Sizes {
    static constexpr int Q_BYTES = A_ROWS * DK * 2, Q_PANEL = A_ROWS * 128;
    static constexpr int K_BYTES = A_TOK * DK * 2, V_BYTES = A_TOK * DV * 2;
    static constexpr int SLOT = K_BYTES > V_BYTES ? K_BYTES : V_BYTES;
    static constexpr int OUT_PITCH = DV * 2 + 16;
    static constexpr int BODY = Q_BYTES + A_SLOTS * SLOT > A_ROWS * OUT_PITCH ? Q_BYTES + A_SLOTS * SLOT : A_ROWS * OUT_PITCH;
    static constexpr int SMEM = BODY + A_NUM_BARS * 8 + 24;
};

template <int DK, int DV, bool SPLIT>
__global__ void __launch_bounds__(A_THREADS, 2) span_attn_kernel(const SpanAttnParams p) {
    using Z = Sizes<DK, DV>;
    extern __shared__ __align__(1024) uint8_t smem[];
    const uint32_t sbase = smem_u32(smem);
    const uint32_t ring = sbase + Z::Q_BYTES;
    const uint32_t full_bar = sbase + Z::BODY;
    const uint32_t empty_bar = full_bar + 8 * A_SLOTS;
    const uint32_t s_full = empty_bar + 8 * A_SLOTS;
    const uint32_t p_full = s_full + 16;
    const uint32_t o_done = p_full + 16;
    const uint32_t q_ready = o_done + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + Z::BODY + A_NUM_BARS * 8);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int G = p.n_kv_heads, group = p.group, H = G * group;
    const int kvh = blockIdx.x % G;
    const int4 blk = __ldg(reinterpret_cast<const int4*>(p.blocks) + blockIdx.x / G);
    const int token0 = blk.y, n_rows = (blk.z - blk.y) * group;
    const int32_t* list = p.path_chunks + __ldg(p.path_off + blk.x);
    const int n_ctx = __ldg(p.positions + blk.z - 1) + 1;
    const int n_tiles = (n_ctx + A_TOK - 1) / A_TOK;
    const int tail = n_ctx - (n_tiles - 1) * A_TOK;  // tokens of the last tile

    if (threadIdx.x == 0) {
        for (int i = 0; i < A_SLOTS; i++) {
            mbar_init(full_bar + 8 * i, 1);
            mbar_init(empty_bar + 8 * i, 1);
        }
        for (int b = 0; b < 2; b++) {
            mbar_init(s_full + 8 * b, 1);
            mbar_init(p_full + 8 * b, 4 * 32);
        }
        mbar_init(o_done, 1);
        mbar_init(q_ready, 4 * 32);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    // Only the stored tokens of the last tile are copied.  The rows behind them meet weights of zero, so they only have to
    // be finite: earlier tiles of this walk are; a slot that has not been used yet is cleared.
    if (tail < A_TOK && n_tiles <= 2) {
        const uint32_t v_slot = ring + ((2 * n_tiles - 1) & (A_SLOTS - 1)) * Z::SLOT;
        for (int i = threadIdx.x; i < Z::V_BYTES / 16; i += A_THREADS) sts128_zero(v_slot + 16 * i);
    }
    fence_proxy_async();
    if (warp == 5) {  // the warp that allocates is the warp that frees
        tmem_alloc(smem_u32(tmem_slot), A_TMEM_COLS);
        tmem_relinquish_alloc_permit();
    }
    tc_fence_before_thread_sync();
    __syncthreads();
    tc_fence_after_thread_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 4) {
        // ---- producer: slot i & 3 takes K of tile i / 2 (even i) or its V (odd i)
        if (lane == 0) {
            int issued = 0;
            for (int i = 0; i < 2 * n_tiles; i++) {
                const int slot = i & (A_SLOTS - 1), use = i / A_SLOTS;
                if (!mbar_wait_bounded(empty_bar + 8 * slot, (use & 1) ^ 1, p.wait_limit)) {
                    report(p.status, STATUS_EMPTY_WAIT_TIMEOUT);
                    break;
                }
                int chunk = __ldg(list + (i >> 1));
                if (chunk < 0 || chunk >= p.max_chunks) {
                    report(p.status, STATUS_BAD_WORK_LIST);  // keep the pipeline moving on a chunk that exists
                    chunk = 0;
                }
                const uint8_t* src = static_cast<const uint8_t*>(p.pool) +
                                     ((size_t)chunk * G + kvh) * (size_t)(Z::K_BYTES + Z::V_BYTES) + ((i & 1) ? Z::K_BYTES : 0);
                const uint32_t dst = ring + slot * Z::SLOT, bar = full_bar + 8 * slot;
                const int panels = (i & 1) ? DV / 64 : DK / 64;
                const bool whole = (i >> 1) < n_tiles - 1 || tail == A_TOK;
                const uint32_t lines = whole ? A_TOK : tail;
                mbar_arrive_expect_tx(bar, panels * lines * 128);
                if (whole) {
                    bulk_copy_g2s(dst, src, panels * A_TOK * 128, bar);
                } else {
                    for (int pn = 0; pn < panels; pn++) bulk_copy_g2s(dst + pn * (A_TOK * 128), src + pn * (A_TOK * 128), lines * 128, bar);
                }
                issued++;
            }
            for (int f = issued > A_SLOTS ? issued - A_SLOTS : 0; f < issued; f++) {
                if (!mbar_wait_bounded(full_bar + 8 * (f & (A_SLOTS - 1)), (f / A_SLOTS) & 1, p.wait_limit)) {
                    report(p.status, STATUS_DRAIN_TIMEOUT);
                    break;
                }
            }
        }
    } else if (warp == 5) {
        // ---- MMA issuer: one thread
        if (elect_one()) {
            bool live = true;
            constexpr uint32_t DESC_HI = umma_desc_sw128_hi(1024);
            constexpr uint32_t IDESC_QK = idesc_bf16(A_ROWS, A_TOK, false), IDESC_PV = idesc_bf16(A_ROWS, DV, true);
            const uint32_t q_lo = umma_desc_sw128_lo(sbase, 16);
            auto issue_qk = [&](int j) {
                const int i = 2 * j, slot = i & (A_SLOTS - 1);
                if (!mbar_wait_bounded(full_bar + 8 * slot, (i / A_SLOTS) & 1, p.wait_limit)) {
                    report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    live = false;
                    return;
                }
                tc_fence_after_thread_sync();
                const uint32_t d = tmem_base + A_COL_S + (j & 1) * A_TOK;
                const uint32_t b_lo = umma_desc_sw128_lo(ring + slot * Z::SLOT, 16);
#pragma unroll
                for (int ks = 0; ks < DK / 16; ks++) {
                    const uint64_t a = umma_desc_pack(q_lo + (((ks >> 2) * Z::Q_PANEL + (ks & 3) * 32) >> 4), DESC_HI);
                    const uint64_t b = umma_desc_pack(b_lo + (((ks >> 2) * (A_TOK * 128) + (ks & 3) * 32) >> 4), DESC_HI);
                    umma_ss_f16(d, a, b, IDESC_QK, ks > 0 ? 1u : 0u);
                }
                umma_commit(s_full + 8 * (j & 1));
                umma_commit(empty_bar + 8 * slot);
            };
            if (!mbar_wait_bounded(q_ready, 0, p.wait_limit)) {
                report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                live = false;
            }
            if (live) issue_qk(0);
            for (int j = 0; j < n_tiles && live; j++) {
                if (j + 1 < n_tiles) issue_qk(j + 1);
                if (!live) break;
                const int i = 2 * j + 1, slot = i & (A_SLOTS - 1);
                if (!mbar_wait_bounded(p_full + 8 * (j & 1), (j >> 1) & 1, p.wait_limit) ||
                    !mbar_wait_bounded(full_bar + 8 * slot, (i / A_SLOTS) & 1, p.wait_limit)) {
                    report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    break;
                }
                tc_fence_after_thread_sync();
                const uint32_t a_tmem = tmem_base + A_COL_S + (j & 1) * A_TOK;  // hi parts, then lo parts, two bf16 per column
                const uint32_t v_lo = umma_desc_sw128_lo(ring + slot * Z::SLOT, A_TOK * 128);
#pragma unroll
                for (int part = 0; part < (SPLIT ? 2 : 1); part++)
#pragma unroll
                    for (int kk = 0; kk < 4; kk++) {
                        const uint64_t b = umma_desc_pack(v_lo + ((kk * 2048) >> 4), DESC_HI);
                        umma_ts_f16(tmem_base, a_tmem + part * 32 + kk * 8, b, IDESC_PV, (j > 0 || kk > 0 || part > 0) ? 1u : 0u);
                    }
                umma_commit(empty_bar + 8 * slot);
                umma_commit(o_done);
            }
        }
    } else {
        // ---- queries -> shared memory, K-major 128-byte-swizzled; rows past the block are zero.  A negative scale is
        // moved into the queries, so that the largest score is the largest product.
        const uint32_t flip = p.scale_log2 < 0.f ? 0x80008000u : 0u;
        constexpr int GR = DK / 8;
        uint4 v[GR];  // all loads of a thread in flight together
#pragma unroll
        for (int u = 0; u < GR; u++) {
            const int i = threadIdx.x + u * (4 * 32), r = i / GR, g = i % GR;
            v[u] = make_uint4(0u, 0u, 0u, 0u);
            if (r < n_rows) {
                const int token = token0 + r / group, head = kvh * group + r % group;
                v[u] = __ldg(reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.q) + ((size_t)token * H + head) * DK) + g);
            }
        }
#pragma unroll
        for (int u = 0; u < GR; u++) {
            const int i = threadIdx.x + u * (4 * 32), r = i / GR, g = i % GR;
            const uint32_t dst = sbase + (g >> 3) * Z::Q_PANEL + r * 128 + (((g & 7) ^ (r & 7)) << 4);
            sts128(dst, (int)(v[u].x ^ flip), (int)(v[u].y ^ flip), (int)(v[u].z ^ flip), (int)(v[u].w ^ flip));
        }
        fence_proxy_async();
        mbar_arrive(q_ready);

        // ---- softmax: thread r owns query row r = TMEM lane r
        const int r = threadIdx.x;
        const bool active = r < n_rows;
        const int my_token = token0 + (active ? r / group : 0);
        const int limit = active ? __ldg(p.positions + my_token) + 1 : 0;
        const int open = __ldg(p.positions + token0) + 1;  // tokens every row of the block sees
        const float scale = fabsf(p.scale_log2);
        const uint32_t lane_addr = tmem_base + ((uint32_t)(warp * 32) << 16);
        float m_used = A_NEG_BIG, l = 0.f;
        bool live = true;
        for (int j = 0; j < n_tiles && live; j++) {
            const int b = j & 1;
            live = mbar_wait_bounded(s_full + 8 * b, (j >> 1) & 1, p.wait_limit);
            live = __all_sync(0xffffffffu, live);
            if (!live) {
                if (lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                break;
            }
            tc_fence_after_thread_sync();
            uint32_t s0[32], s1[32];
            tmem_ld32(lane_addr + A_COL_S + b * A_TOK, s0);
            tmem_ld32(lane_addr + A_COL_S + b * A_TOK + 32, s1);
            tmem_wait_ld();
            if ((j + 1) * A_TOK > open) {
                const int seen = limit - j * A_TOK;
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    if (i >= seen) s0[i] = 0xff800000u;
                    if (32 + i >= seen) s1[i] = 0xff800000u;
                }
            }
            float alpha = 1.f;
            bool rescale = false;
            {
                float mx = fmaxf(__uint_as_float(s0[0]), __uint_as_float(s1[0]));
#pragma unroll
                for (int i = 1; i < 32; i++) mx = fmaxf(mx, fmaxf(__uint_as_float(s0[i]), __uint_as_float(s1[i])));
                mx = fmaxf(mx * scale, A_NEG_BIG);
                if (scale == 0.f) mx = 0.f;  // 0 * -inf above
                if (j == 0) {
                    m_used = mx;
                } else if (mx > m_used + A_RESCALE_STEP) {
                    alpha = fast_exp2(m_used - mx);
                    m_used = mx;
                    l *= alpha;
                    rescale = true;
                }
            }
            float sum = 0.f;
#pragma unroll
            for (int i = 0; i < 32; i++) {
                s0[i] = __float_as_uint(fast_exp2(fmaf(__uint_as_float(s0[i]), scale, -m_used)));
                s1[i] = __float_as_uint(fast_exp2(fmaf(__uint_as_float(s1[i]), scale, -m_used)));
                sum += __uint_as_float(s0[i]) + __uint_as_float(s1[i]);
            }
            l += sum;
            uint32_t pk[32];
#pragma unroll
            for (int i = 0; i < 16; i++) {
                pk[i] = pack_bf16(__uint_as_float(s0[2 * i]), __uint_as_float(s0[2 * i + 1]));
                pk[16 + i] = pack_bf16(__uint_as_float(s1[2 * i]), __uint_as_float(s1[2 * i + 1]));
            }
            tmem_st32(lane_addr + A_COL_S + b * A_TOK, pk);
            if (SPLIT) {
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    pk[i] = pack_bf16(__uint_as_float(s0[2 * i]) - __uint_as_float(pk[i] << 16),
                                      __uint_as_float(s0[2 * i + 1]) - __uint_as_float(pk[i] & 0xffff0000u));
                    pk[16 + i] = pack_bf16(__uint_as_float(s1[2 * i]) - __uint_as_float(pk[16 + i] << 16),
                                           __uint_as_float(s1[2 * i + 1]) - __uint_as_float(pk[16 + i] & 0xffff0000u));
                }
                tmem_st32(lane_addr + A_COL_S + b * A_TOK + 32, pk);
            }
            if (j > 0) {
                // O += P V of tile j - 1 is complete (every thread follows o_done phase by phase)
                live = mbar_wait_bounded(o_done, (j - 1) & 1, p.wait_limit);
                live = __all_sync(0xffffffffu, live);
                if (!live) {
                    if (lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    break;
                }
            }
            if (__any_sync(0xffffffffu, rescale)) {
                tc_fence_after_thread_sync();
#pragma unroll
                for (int c = 0; c < DV / 32; c++) {
                    uint32_t o[32];
                    tmem_ld32(lane_addr + c * 32, o);
                    tmem_wait_ld();
#pragma unroll
                    for (int i = 0; i < 32; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
                    tmem_st32(lane_addr + c * 32, o);
                }
            }
            tmem_wait_st();
            tc_fence_before_thread_sync();
            mbar_arrive(p_full + 8 * b);
        }
        if (live) {
            live = mbar_wait_bounded(o_done, (n_tiles - 1) & 1, p.wait_limit);
            live = __all_sync(0xffffffffu, live);
            if (!live && lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
        }
        if (live) {
            tc_fence_after_thread_sync();
            // ---- epilogue: the sink has score 0; rows leave as bf16 through shared memory (every MMA has completed, so
            // queries and ring are free), each warp its own 32 rows
            float inv;
            {
                float total = l;
                float M = m_used;
                if (p.sink) {
                    M = fmaxf(m_used, 0.f);
                    total = l * fast_exp2(m_used - M) + fast_exp2(-M);
                }
                inv = total > 0.f ? fast_exp2(m_used - M) / total : 0.f;
            }
            const float pos = (float)(limit - 1);
#pragma unroll
            for (int c = 0; c < DV / 32; c++) {
                uint32_t o[32];
                tmem_ld32(lane_addr + c * 32, o);
                tmem_wait_ld();
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    float a = __uint_as_float(o[2 * i]) * inv, bb = __uint_as_float(o[2 * i + 1]) * inv;
                    if (p.value_freq) {
                        float sn, cs;
                        fast_sincos(pos * __ldg(p.value_freq + c * 16 + i), &sn, &cs);
                        const float t = a * cs + bb * sn;
                        bb = bb * cs - a * sn;
                        a = t;
                    }
                    o[i] = pack_bf16(a, bb);
                }
#pragma unroll
                for (int i = 0; i < 4; i++)
                    *reinterpret_cast<uint4*>(smem + r * Z::OUT_PITCH + c * 64 + 16 * i) = make_uint4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]);
            }
            __syncwarp();
            constexpr int LPR = DV / 8;  // lanes per row, 16 bytes each
            const int rows_here = min(32, n_rows - warp * 32);
            for (int rr = lane / LPR; rr < rows_here; rr += 32 / LPR) {
                const int row = warp * 32 + rr, token = token0 + row / group, head = kvh * group + row % group;
                const uint4 v = *reinterpret_cast<const uint4*>(smem + row * Z::OUT_PITCH + 16 * (lane % LPR));
                *(reinterpret_cast<uint4*>(static_cast<__nv_bfloat16*>(p.out) + ((size_t)token * H + head) * DV) + lane % LPR) = v;
            }
        }
    }
    // ---- common exit: nobody touches TMEM after this barrier, then the allocating warp frees it
    tc_fence_before_thread_sync();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after_thread_sync();
        tmem_dealloc(tmem_base, A_TMEM_COLS);
    }
}

template <int DK, int DV>
cudaError_t launch(const SpanAttnParams& p, cudaStream_t stream) {
    auto* k = p.split_weights ? span_attn_kernel<DK, DV, true> : span_attn_kernel<DK, DV, false>;
    constexpr int smem = Sizes<DK, DV>::SMEM;
    static_assert(2 * (smem + 1024) <= 233472, "two CTAs do not fit in one SM's shared memory");
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    if (e != cudaSuccess) return e;
    k<<<p.n_blocks * p.n_kv_heads, A_THREADS, smem, stream>>>(p);
    return cudaGetLastError();
}

}  // namespace

bool span_attn_serves(const Geometry& g, int d_value, int block_query_rows) {
    return g.esize == 2 && g.chunk_size == A_TOK && (g.d_head == 64 || g.d_head == 128) && (g.d_value == 64 || g.d_value == 128) &&
           g.d_value == d_value && block_query_rows <= A_ROWS;
}

cudaError_t launch_span_attn(const SpanAttnParams& p, int d_key, int d_value, cudaStream_t stream) {
    if (d_key == 128) return d_value == 128 ? launch<128, 128>(p, stream) : launch<128, 64>(p, stream);
    return d_value == 128 ? launch<64, 128>(p, stream) : launch<64, 64>(p, stream);
}

}  // namespace ca
