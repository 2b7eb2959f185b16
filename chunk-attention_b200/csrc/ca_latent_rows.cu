// Attention over a latent cache on the Blackwell tensor path (bf16, tcgen05): decode items of the planner's work list, and
// portions of prompts where expanding the latents into per-head keys and values (ca_latent_span.cu) does not pay.
//
// A token's pool row is key and value of every head at once, so the query heads of a token, and the tokens of a block, are
// rows of ONE product against the rows staged in shared memory: row r is head r % H of token r / H.  There are few of them
// (up to 64) and the values are long, so the products are formed transposed, cache rows and value elements on the M side:
//   S^T = K Q^T   two 64-element panels at a time: M = 64 tokens of one panel and the same 64 of the next, N = query rows of one
//                 panel and of the next; the blocks on the diagonal of D are the two panels' shares of the scores (the others
//                 are not used).  D in TMEM, two buffers, so that tile j + 1 is scored under the softmax of tile j
//   softmax       the shares go through shared memory once, so that 256 / N threads share a query row; fp32, log2 units;
//                 every row has a window.  O is rescaled only when a row's maximum has grown by more than 8.  The
//                 weights go back to shared memory as bf16 hi + lo parts, whose sum has 16 bits of the fp32 weight
//   O^T += V^T P^T  M = 128 value elements (one TMEM block each), N = hi and lo parts of the query rows (up to 32 rows: side by
//                 side in one product; 64: one after the other); A = the same staged rows read the other way
// Cache rows arrive by 1-D TMA bulk copies, verbatim (the pool's lines are the swizzled operand layout), in a ring of
// 16 KiB units: two 64-element panels of a 64-token chunk, released one by one as the second product has used them.  Decode
// emits one partial per row and item, combined by a merge kernel; portions emit finished rows.
// Warp roles: 0-7 softmax and epilogue, 8 TMA producer, 9 TMEM and the first product's issue, 10 the second one's.
//
// Every wait is bounded: on expiry a status code is recorded, every role runs out without waiting further, nothing is
// stored, and the TMEM columns are freed at the common exit.
#include <algorithm>

#include "ca_kernels.h"
#include "ca_plan.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int L_PITCH = 68;                           // floats between score rows
constexpr int L_SOFT = 256, L_THREADS = L_SOFT + 96,  // softmax threads, and all
              L_TOK = 64, L_PANEL = L_TOK * 128, L_UNIT = 2 * L_PANEL, L_MAX_UNITS = 16, L_MAX_ROWS = 64;
constexpr float L_NEG_BIG = -1.0e30f, L_LOG2E = 1.4426950408889634f, L_RESCALE_STEP = 8.f;

__host__ __device__ constexpr uint32_t idesc_bf16(int m, int n, bool a_mn_major) { return umma_idesc_f16(m, n, a_mn_major, false) | (1u << 7) | (1u << 10); }
__device__ __forceinline__ void report(int* status, int code) { atomicCAS(status, STATUS_OK, code); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ void softmax_warps_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void sts64(uint32_t addr, uint32_t x, uint32_t y) { asm volatile("st.shared.v2.u32 [%0], {%1,%2};" ::"r"(addr), "r"(x), "r"(y) : "memory"); }

template <int N> __device__ __forceinline__ void tmem_ld(uint32_t taddr, uint32_t (&r)[N]);
template <> __device__ __forceinline__ void tmem_ld<16>(uint32_t taddr, uint32_t (&r)[16]) { tmem_ld16(taddr, r); }
template <> __device__ __forceinline__ void tmem_ld<32>(uint32_t taddr, uint32_t (&r)[32]) { tmem_ld32(taddr, r); }

// byte offsets of the parts of shared memory behind the ring
struct Layout {
    int units, q, weights, scores, end;
};
template <int N> __host__ __device__ inline Layout layout_of(int gpr, int units) {
    Layout l;
    l.units = units;
    l.q = units * L_UNIT;                        // queries: [gpr / 8 panels][N lines of 128 bytes]
    l.weights = l.q + N * gpr * 16;              // weights: hi and lo, [N lines of 64 tokens] each
    l.scores = l.weights + 2 * N * 128;          // fp32 [2 shares][N][L_PITCH]
    l.end = l.scores + 2 * N * L_PITCH * 4;
    return l;
}

template <int N, bool SPAN>
__global__ void __launch_bounds__(L_THREADS) latent_rows_kernel(const LatentParams p, int units) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int TPR = L_SOFT / N, PER = L_TOK / TPR;  // threads of a row, tokens of a thread
    constexpr int CH = N < 32 ? N : 32;              // TMEM columns read at a time
    constexpr bool WIDE = N <= 32;                   // hi and lo weights in one product
    constexpr uint32_t DESC_HI = umma_desc_sw128_hi(1024);
    constexpr int S_COLS = 2 * N, O_COLS = WIDE ? 2 * N : N;
    const int gpr = p.geo.gpr, panels = gpr >> 3, tile_units = (panels + 1) >> 1, blocks = (p.geo.d_value + 127) >> 7;
    const Layout lay = layout_of<N>(gpr, units);
    const uint32_t sbase = smem_u32(smem);
    const uint32_t q_base = sbase + lay.q, w_base = sbase + lay.weights;
    float* const sc = reinterpret_cast<float*>(smem + lay.scores);
    uint64_t* const bar_mem = reinterpret_cast<uint64_t*>(smem + lay.end);
    const uint32_t full = smem_u32(bar_mem), empty = full + 8 * L_MAX_UNITS, s_full = empty + 8 * L_MAX_UNITS, p_full = s_full + 16,
                   o_done = p_full + 8, q_ready = o_done + 8, s_empty = q_ready + 8;
    float* const alpha_s = reinterpret_cast<float*>(bar_mem + 2 * L_MAX_UNITS + 7);  // [N]
    int* const flag_s = reinterpret_cast<int*>(alpha_s + L_MAX_ROWS);                 // [2]
    uint32_t* const tmem_slot = reinterpret_cast<uint32_t*>(flag_s + 2);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int H = p.n_heads;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");  // the merge kernel may be set up; it waits for this one's end

    // ---- the block of rows and its tokens: [start, end) relative to position `first` of list[0]
    int token0, n_rows, first, end, low, row_lo = (int)blockIdx.y * N, slot_base = 0;
    const int32_t* list;
    if (SPAN) {
        const int4 b = reinterpret_cast<const int4*>(p.blocks)[blockIdx.x];
        token0 = b.y;
        n_rows = (b.z - b.y) * H;
        if (row_lo >= n_rows) return;
        n_rows = min(N, n_rows - row_lo);
        first = 0;
        list = p.path_chunks + p.path_off[b.x];
        end = p.positions[token0 + (row_lo + n_rows - 1) / H] + 1;
        low = p.positions[token0 + row_lo / H];
    } else {
        const int4* it = p.items + 4 * blockIdx.x;
        const int4 a = __ldg(it), b = __ldg(it + 1);  // tiles, first, row, rows | slot, flags, last, chunks ...
        token0 = a.z;
        n_rows = a.w * H;
        if (row_lo >= n_rows) return;
        n_rows = min(N, n_rows - row_lo);
        first = a.y;
        slot_base = b.x;
        list = reinterpret_cast<const int32_t*>(it) + 7;
        end = (a.x - 1) * L_TOK + min(L_TOK, b.z + ((b.y & ITEM_FLAG_TAIL) ? p.delta_tokens : 0));
        low = p.positions[token0];
        for (int i = 1; i < a.w; i++) low = min(low, p.positions[token0 + i]);
    }
    const int start = p.window > 0 ? max(0, low - p.window + 1 - first) / L_TOK * L_TOK : 0;
    const int n_tiles = end > start ? (end - start + L_TOK - 1) / L_TOK : 0;
    const int tail = end - start - (n_tiles - 1) * L_TOK;  // tokens of the last tile

    if (tid == 0) {
        for (int i = 0; i < units; i++) {
            mbar_init(full + 8 * i, 1);
            mbar_init(empty + 8 * i, 1);
        }
        mbar_init(s_full, 1);
        mbar_init(s_full + 8, 1);
        mbar_init(p_full, L_SOFT);
        mbar_init(o_done, 1);
        mbar_init(q_ready, L_SOFT);
        mbar_init(s_empty, L_SOFT / 32);
        mbar_init(s_empty + 8, L_SOFT / 32);
        flag_s[0] = flag_s[1] = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    // Only the stored tokens of the last tile are copied.  The lines behind them meet weights of zero, so they only have to be
    // finite: they are cleared in the units that tile will use (what earlier tiles bring there is finite, too).
    if (n_tiles > 0 && tail < L_TOK) {
        const int lines = L_TOK - tail;
        for (int i = tid; i < tile_units * 2 * lines * 8; i += L_THREADS) {
            const int pn = i / (lines * 8), q = i % (lines * 8);
            const int unit = ((n_tiles - 1) * tile_units + (pn >> 1)) % units;
            sts128_zero(sbase + unit * L_UNIT + (pn & 1) * L_PANEL + tail * 128 + q * 16);
        }
        fence_proxy_async();
    }
    constexpr uint32_t COL_S = 4 * O_COLS;  // O blocks at columns 0, O_COLS, ...
    constexpr uint32_t COLS = 2 * S_COLS + COL_S <= 256 ? 256 : 512;
    static_assert(2 * S_COLS + COL_S <= 512, "tensor memory");
    if (warp == 9) {  // the warp that allocates is the warp that frees
        tmem_alloc(smem_u32(tmem_slot), COLS);
        tmem_relinquish_alloc_permit();
    }
    tc_fence_before_thread_sync();
    __syncthreads();
    tc_fence_after_thread_sync();
    const uint32_t tmem_base = *tmem_slot;

    if (warp == 8) {
        // ---- producer
        if (lane == 0) {
            int issued = 0, slot = 0, parity = 1;
            bool live = true;
            for (int j = 0; j < n_tiles && live; j++) {
                const int at = start + j * L_TOK;
                const uint32_t bytes = min(L_TOK, end - at) * 128;
                int chunk = __ldg(list + at / L_TOK);
                if (chunk < 0 || chunk >= p.max_chunks) {
                    report(p.status, STATUS_BAD_WORK_LIST);
                    chunk = 0;
                }
                const uint8_t* src = static_cast<const uint8_t*>(p.pool) + (size_t)chunk * (L_TOK * 16) * gpr;
                for (int u = 0; u < tile_units; u++, issued++) {
                    if (!mbar_wait_bounded(empty + 8 * slot, parity, p.wait_limit)) {
                        report(p.status, STATUS_EMPTY_WAIT_TIMEOUT);
                        live = false;
                        break;
                    }
                    const bool two = 2 * u + 1 < panels;
                    const uint32_t dst = sbase + slot * L_UNIT, bar = full + 8 * slot;
                    mbar_arrive_expect_tx(bar, two ? 2 * bytes : bytes);
                    if (two && bytes == L_PANEL) {
                        bulk_copy_g2s(dst, src + 2 * u * L_PANEL, 2 * L_PANEL, bar);
                    } else {
                        bulk_copy_g2s(dst, src + 2 * u * L_PANEL, bytes, bar);
                        if (two) bulk_copy_g2s(dst + L_PANEL, src + (2 * u + 1) * L_PANEL, bytes, bar);
                    }
                    if (++slot == units) {
                        slot = 0;
                        parity ^= 1;
                    }
                }
            }
            for (int f = issued > units ? issued - units : 0; f < issued; f++) {
                if (!mbar_wait_bounded(full + 8 * (f % units), (f / units) & 1, p.wait_limit)) {
                    report(p.status, STATUS_DRAIN_TIMEOUT);
                    break;
                }
            }
        }
    } else if (warp == 9) {
        // ---- scores: one thread issues, unit by unit as a tile's rows arrive, up to two tiles ahead of the softmax
        if (elect_one()) {
            constexpr uint32_t IDESC_QK2 = idesc_bf16(128, 2 * N, false), IDESC_QK1 = idesc_bf16(128, N, false);
            bool live = true;
            auto wait = [&](uint32_t bar, int parity) {
                if (live && !mbar_wait_bounded(bar, parity, p.wait_limit)) {
                    report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    live = false;
                }
            };
            const uint32_t q_lo = umma_desc_sw128_lo(q_base, 16);
            int slot = 0, parity = 0;
            wait(q_ready, 0);
            for (int j = 0; j < n_tiles && live; j++) {
                if (j >= 2) wait(s_empty + 8 * (j & 1), ((j >> 1) - 1) & 1);
                const uint32_t d = tmem_base + COL_S + (j & 1) * S_COLS;
                uint32_t b_lo = q_lo;
                for (int u = 0; u < tile_units; u++) {
                    wait(full + 8 * slot, parity);
                    if (!live) break;
                    tc_fence_after_thread_sync();
                    const uint32_t a_lo = umma_desc_sw128_lo(sbase + slot * L_UNIT, 16);
                    // a last panel without a partner: its share only (the lower half of D is not used)
                    const uint32_t idesc = 2 * u + 1 < panels ? IDESC_QK2 : IDESC_QK1;
                    umma_ss_f16(d, umma_desc_pack(a_lo, DESC_HI), umma_desc_pack(b_lo, DESC_HI), idesc, u > 0 ? 1u : 0u);
#pragma unroll
                    for (int ks = 1; ks < 4; ks++)
                        umma_ss_f16(d, umma_desc_pack(a_lo + 2 * ks, DESC_HI), umma_desc_pack(b_lo + 2 * ks, DESC_HI), idesc, 1u);
                    if (u >= blocks) umma_commit(empty + 8 * slot);  // holds no values
                    b_lo += 2 * N * 8;
                    if (++slot == units) {
                        slot = 0;
                        parity ^= 1;
                    }
                }
                if (live) umma_commit(s_full + 8 * (j & 1));
            }
        }
    } else if (warp == 10) {
        // ---- the second product: one thread issues, and frees the units block by block
        if (elect_one()) {
            constexpr uint32_t IDESC_PV = idesc_bf16(128, O_COLS, true);
            const uint32_t p_lo = umma_desc_sw128_lo(w_base, 16);
            int slot = 0;
            for (int j = 0; j < n_tiles; j++) {
                if (!mbar_wait_bounded(p_full, j & 1, p.wait_limit)) {
                    report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                    break;
                }
                tc_fence_after_thread_sync();
                for (int m = 0; m < tile_units; m++) {
                    if (m < blocks) {
                        const uint32_t d = tmem_base + m * O_COLS;
                        const uint32_t a_lo = umma_desc_sw128_lo(sbase + slot * L_UNIT, L_PANEL);
#pragma unroll
                        for (int part = 0; part < (WIDE ? 1 : 2); part++)
#pragma unroll
                            for (int kk = 0; kk < 4; kk++)
                                umma_ss_f16(d, umma_desc_pack(a_lo + 128 * kk, DESC_HI), umma_desc_pack(p_lo + part * (N * 8) + 2 * kk, DESC_HI), IDESC_PV,
                                            part + kk > 0 ? 1u : (j > 0 ? 1u : 0u));
                        umma_commit(empty + 8 * slot);
                    }
                    if (++slot == units) slot = 0;
                }
                umma_commit(o_done);
            }
        }
    } else {
        // ---- queries: latent part as it comes, shared part turned by the row's position, zeros up to the pool's row.  Loads
        // are requested in batches before any of them is used
        {
            const __nv_bfloat16* q_lat = static_cast<const __nv_bfloat16*>(p.q_lat) + ((size_t)token0 * H + row_lo) * p.kv_rank;  // rows follow one another
            const __nv_bfloat16* q_rot = static_cast<const __nv_bfloat16*>(p.q_rot);
            const int half = p.rot / 2;
            auto line = [&](int r, int g) { return q_base + (g >> 3) * (N * 128) + r * 128 + (((g & 7) ^ (r & 7)) << 4); };
            auto aligned = [](const void* x) { return reinterpret_cast<uintptr_t>(x) % 16 == 0; };
            const bool whole = p.kv_rank % 8 == 0 && aligned(p.q_lat);
            const bool pairs = whole && half % 8 == 0 && half > 0 && p.q_rot_row % 8 == 0 && p.q_rot_head % 8 == 0 && aligned(p.q_rot) && aligned(p.freq);
            const int done_g = whole ? p.kv_rank / 8 : 0;  // granules below it hold latent elements only
            constexpr int AHEAD = 8;
            uint4 v[AHEAD];
#pragma unroll
            for (int k = 0; k < AHEAD; k++) {
                const int i = tid + L_SOFT * k;
                v[k] = make_uint4(0u, 0u, 0u, 0u);
                if (i < n_rows * done_g) v[k] = __ldg(reinterpret_cast<const uint4*>(q_lat) + i);
            }
            if (pairs) {  // a granule of the rotated part's first half and its partner in the second
                const int units_r = half / 8;
                for (int i = tid; i < N * units_r; i += L_SOFT) {
                    const int r = i / units_r, u = i % units_r, rr = row_lo + r, token = token0 + rr / H;
                    uint4 a = make_uint4(0u, 0u, 0u, 0u), b = a;
                    if (r < n_rows) {
                        const uint4* src = reinterpret_cast<const uint4*>(q_rot + (size_t)token * p.q_rot_row + (size_t)(rr % H) * p.q_rot_head);
                        a = __ldg(src + u);
                        b = __ldg(src + units_r + u);
                        const float pos = (float)p.positions[token];
                        const float4 f0 = *reinterpret_cast<const float4*>(p.freq + 8 * u), f1 = *reinterpret_cast<const float4*>(p.freq + 8 * u + 4);
                        const float f[8] = {f0.x, f0.y, f0.z, f0.w, f1.x, f1.y, f1.z, f1.w};
                        uint32_t* aw = reinterpret_cast<uint32_t*>(&a);
                        uint32_t* bw = reinterpret_cast<uint32_t*>(&b);
#pragma unroll
                        for (int k = 0; k < 4; k++) {
                            const float x0 = __uint_as_float(aw[k] << 16), x1 = __uint_as_float(aw[k] & 0xffff0000u);
                            const float y0 = __uint_as_float(bw[k] << 16), y1 = __uint_as_float(bw[k] & 0xffff0000u);
                            float s0, c0, s1, c1;
                            fast_sincos(pos * f[2 * k], &s0, &c0);
                            fast_sincos(pos * f[2 * k + 1], &s1, &c1);
                            aw[k] = pack_bf16(x0 * c0 - y0 * s0, x1 * c1 - y1 * s1);
                            bw[k] = pack_bf16(y0 * c0 + x0 * s0, y1 * c1 + x1 * s1);
                        }
                    }
                    sts128(line(r, done_g + u), (int)a.x, (int)a.y, (int)a.z, (int)a.w);
                    sts128(line(r, done_g + units_r + u), (int)b.x, (int)b.y, (int)b.z, (int)b.w);
                }
                const int behind = gpr - done_g - 2 * units_r;
                for (int i = tid; i < N * behind; i += L_SOFT) sts128_zero(line(i / behind, done_g + 2 * units_r + i % behind));
            }
            if (done_g > 0) {
                const int step_r = L_SOFT / done_g, step_g = L_SOFT % done_g;
                int r = tid / done_g, g = tid % done_g;
                for (int i0 = tid; i0 < N * done_g; i0 += L_SOFT * AHEAD) {
#pragma unroll
                    for (int k = 0; k < AHEAD; k++) {
                        if (r < N) sts128(line(r, g), (int)v[k].x, (int)v[k].y, (int)v[k].z, (int)v[k].w);
                        r += step_r;
                        g += step_g;
                        if (g >= done_g) {
                            g -= done_g;
                            r++;
                        }
                    }
#pragma unroll
                    for (int k = 0; k < AHEAD; k++) {
                        const int i = i0 + L_SOFT * (AHEAD + k);
                        v[k] = make_uint4(0u, 0u, 0u, 0u);
                        if (i < n_rows * done_g) v[k] = __ldg(reinterpret_cast<const uint4*>(q_lat) + i);
                    }
                }
            }
            if (!pairs) {  // any sizes, element by element
                const int rest = gpr - done_g;
                for (int i = tid; i < N * rest; i += L_SOFT) {
                    const int r = i / rest, g = done_g + i % rest, rr = row_lo + r, token = token0 + rr / H;
                    float x[8];
#pragma unroll
                    for (int k = 0; k < 8; k++) {
                        const int e = 8 * g + k, d = e - p.kv_rank;
                        x[k] = 0.f;
                        if (r >= n_rows) continue;
                        if (d < 0) {
                            x[k] = __bfloat162float(q_lat[(size_t)r * p.kv_rank + e]);
                        } else if (d < p.rot) {
                            const __nv_bfloat16* qr = q_rot + (size_t)token * p.q_rot_row + (size_t)(rr % H) * p.q_rot_head;
                            const int pair = d < half ? d : d - half;
                            float sn, cs;
                            fast_sincos((float)p.positions[token] * __ldg(p.freq + pair), &sn, &cs);
                            const float a = __bfloat162float(qr[pair]), b = __bfloat162float(qr[pair + half]);
                            x[k] = d < half ? a * cs - b * sn : b * cs + a * sn;
                        }
                    }
                    sts128(line(r, g), (int)pack_bf16(x[0], x[1]), (int)pack_bf16(x[2], x[3]), (int)pack_bf16(x[4], x[5]), (int)pack_bf16(x[6], x[7]));
                }
            }
            fence_proxy_async();
            mbar_arrive(q_ready);
        }

        // ---- softmax: thread tid has PER tokens of row tid / TPR: fours of tokens, TPR threads side by side
        const int row = tid / TPR, part = tid % TPR, shares = panels > 1 ? 2 : 1, quarter = warp & 3, side = warp >> 2;
        int lo = 0, hi = 0;  // what the row sees, relative to `first`
        if (row < n_rows) {
            const int pos = p.positions[token0 + (row_lo + row) / H] - first;
            hi = min(pos + 1, end);
            lo = p.window > 0 ? pos - p.window + 1 : 0;
        }
        const float scale = fabsf(p.scale_log2), sign = p.scale_log2 < 0.f ? -1.f : 1.f;
        const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16);
        float m_used = L_NEG_BIG, l = 0.f;
        bool live = true;
        for (int j = 0; j < n_tiles; j++) {
            const int b = j & 1, at = start + j * L_TOK;
            // a wait that has run out lets everything run through without waiting: the warps keep meeting at their barriers
            if (live) {
                live = mbar_wait_bounded(s_full + 8 * b, (j >> 1) & 1, p.wait_limit);
                live = __all_sync(0xffffffffu, live);
                if (!live && lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
            }
            tc_fence_after_thread_sync();
            // lane = token of a share: quarters 0 and 1 of the lanes the first panels', columns 0 .., quarters 2 and 3 the second
            // ones', columns N ..; the two warps of a quarter take half of the columns each
            if ((shares == 2 || quarter < 2) && (N >= 32 || side == 0)) {
                constexpr int SC = N >= 32 ? N / 2 : N;
                float* const mine = sc + ((quarter >> 1) * N + side * SC) * L_PITCH + (quarter & 1) * 32 + lane;
                uint32_t s[SC];
                tmem_ld<SC>(lane_addr + COL_S + b * S_COLS + (quarter >> 1) * N + side * SC, s);
                tmem_wait_ld();
#pragma unroll
                for (int i = 0; i < SC; i++) mine[i * L_PITCH] = __uint_as_float(s[i]);
            }
            tc_fence_before_thread_sync();
            __syncwarp();
            if (lane == 0) mbar_arrive(s_empty + 8 * b);
            softmax_warps_sync();
            if (tid == 0) flag_s[b ^ 1] = 0;  // everyone has read it in the tile before
            float x[PER];
            float mx = -INFINITY;
#pragma unroll
            for (int i = 0; i < PER / 4; i++) {
                const int t = (i * TPR + part) * 4;
                const float4 v = *reinterpret_cast<const float4*>(sc + row * L_PITCH + t);
                float in[4] = {v.x, v.y, v.z, v.w};
                if (shares == 2) {
                    const float4 w = *reinterpret_cast<const float4*>(sc + (N + row) * L_PITCH + t);
                    in[0] += w.x;
                    in[1] += w.y;
                    in[2] += w.z;
                    in[3] += w.w;
                }
#pragma unroll
                for (int k = 0; k < 4; k++) x[4 * i + k] = in[k] * sign;
            }
            if (at < lo || at + L_TOK > hi) {
#pragma unroll
                for (int i = 0; i < PER; i++) {
                    const int c = at + ((i >> 2) * TPR + part) * 4 + (i & 3);
                    if (c < lo || c >= hi) x[i] = -INFINITY;
                }
            }
#pragma unroll
            for (int i = 0; i < PER; i++) mx = fmaxf(mx, x[i]);
#pragma unroll
            for (int o = 1; o < TPR; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            mx = scale == 0.f ? 0.f : fmaxf(mx * scale, L_NEG_BIG);
            float alpha = 1.f;
            if (j == 0) {
                m_used = mx;
            } else if (mx > m_used + L_RESCALE_STEP) {
                alpha = fast_exp2(m_used - mx);
                m_used = mx;
                l *= alpha;
                flag_s[b] = 1;
            }
            if (part == 0) alpha_s[row] = alpha;
            softmax_warps_sync();
            if (j > 0) {
                // the second product of tile j - 1 is complete: O may be rescaled and the weights replaced
                if (live) {
                    live = mbar_wait_bounded(o_done, (j - 1) & 1, p.wait_limit);
                    live = __all_sync(0xffffffffu, live);
                    if (!live && lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
                }
                if (*reinterpret_cast<volatile int*>(flag_s + b)) {
                    tc_fence_after_thread_sync();
                    for (int m = side; m < blocks; m += 2)
#pragma unroll
                        for (int c = 0; c < O_COLS; c += CH) {
                            uint32_t o[CH];
                            tmem_ld<CH>(lane_addr + m * O_COLS + c, o);
                            tmem_wait_ld();
#pragma unroll
                            for (int i = 0; i < CH; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha_s[(c + i) % N]);
                            if constexpr (CH == 32) tmem_st32(lane_addr + m * O_COLS + c, o);
                            else tmem_st16(lane_addr + m * O_COLS + c, o);
                        }
                    tmem_wait_st();
                }
            }
#pragma unroll
            for (int i = 0; i < PER / 4; i++) {
                const int t = (i * TPR + part) * 4;
                float e[4];
#pragma unroll
                for (int k = 0; k < 4; k++) {
                    e[k] = x[4 * i + k] == -INFINITY ? 0.f : fast_exp2(fmaf(x[4 * i + k], scale, -m_used));
                    l += e[k];
                }
                const uint32_t h0 = pack_bf16(e[0], e[1]), h1 = pack_bf16(e[2], e[3]);
                const uint32_t l0 = pack_bf16(e[0] - __uint_as_float(h0 << 16), e[1] - __uint_as_float(h0 & 0xffff0000u));
                const uint32_t l1 = pack_bf16(e[2] - __uint_as_float(h1 << 16), e[3] - __uint_as_float(h1 & 0xffff0000u));
                const uint32_t dst = w_base + row * 128 + (((t >> 3) ^ (row & 7)) << 4) + (t & 4) * 2;
                sts64(dst, h0, h1);
                sts64(dst + N * 128, l0, l1);
            }
            fence_proxy_async();
            tc_fence_before_thread_sync();
            mbar_arrive(p_full);
        }
        if (n_tiles > 0 && live) {
            live = mbar_wait_bounded(o_done, (n_tiles - 1) & 1, p.wait_limit);
            live = __all_sync(0xffffffffu, live);
            if (!live && lane == 0) report(p.status, STATUS_FULL_WAIT_TIMEOUT);
        }
        tc_fence_after_thread_sync();
        // ---- epilogue: the factor of every row through shared memory, then lane = value element, column = row
#pragma unroll
        for (int o = 1; o < TPR; o <<= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
        if (part == 0) {
            const int rr = row_lo + row, head = rr % H;
            float f = 1.f;
            if (SPAN) {
                float total = l, M = m_used;
                if (p.sink && row < n_rows) {
                    const float sk = p.sink[head] * L_LOG2E;
                    M = fmaxf(m_used, sk);
                    total = l * fast_exp2(m_used - M) + fast_exp2(sk - M);
                }
                f = total > 0.f ? fast_exp2(m_used - M) / total : 0.f;
            } else if (row < n_rows && live) {
                p.part_ml[((size_t)slot_base + rr / H) * H + head] = make_float2(m_used, l);
            }
            alpha_s[row] = f;
        }
        softmax_warps_sync();
        if (live) {
            for (int m = side; m < blocks; m += 2) {
                const int e = m * 128 + quarter * 32 + lane;
                // rows are consecutive (token, head) pairs
                __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + ((size_t)token0 * H + row_lo) * p.kv_rank + e;
                float* part_o = p.part_o + ((size_t)slot_base * H + row_lo) * p.part_width + e;
#pragma unroll
                for (int c = 0; c < N; c += CH) {
                    uint32_t o[CH];
                    if (n_tiles > 0) {
                        tmem_ld<CH>(lane_addr + m * O_COLS + c, o);
                        tmem_wait_ld();
                        if (WIDE) {
                            uint32_t o2[CH];
                            tmem_ld<CH>(lane_addr + m * O_COLS + N + c, o2);
                            tmem_wait_ld();
#pragma unroll
                            for (int i = 0; i < CH; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) + __uint_as_float(o2[i]));
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < CH; i++) o[i] = 0u;
                    }
                    if (SPAN) {
                        if (e < p.kv_rank)
#pragma unroll
                            for (int i = 0; i < CH; i++, out += p.kv_rank)
                                if (c + i < n_rows) *out = __float2bfloat16_rn(__uint_as_float(o[i]) * alpha_s[c + i]);
                    } else if (e < p.part_width) {
#pragma unroll
                        for (int i = 0; i < CH; i++, part_o += p.part_width)
                            if (c + i < n_rows) *part_o = __uint_as_float(o[i]);
                    }
                }
            }
        }
    }
    // ---- common exit: nobody touches TMEM after this barrier, then the allocating warp frees it
    tc_fence_before_thread_sync();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after_thread_sync();
        tmem_dealloc(tmem_base, COLS);
    }
}

// One CTA per (row, query head), four value elements per thread: combines the row's partials and the sink, stores bf16.
__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentParams p) {
    const int H = p.n_heads, row = blockIdx.x / H, head = blockIdx.x % H, e = threadIdx.x * 4;
    const int b = p.merge_off[row], n = p.merge_off[row + 1] - b;
    asm volatile("griddepcontrol.wait;" ::: "memory");  // what comes before is not written by the kernel before this one
    constexpr int AHEAD = 4;
    const bool on = e < p.part_width;
    float M = L_NEG_BIG, L = 0.f, acc[4] = {0.f, 0.f, 0.f, 0.f};
    if (p.sink) {
        M = p.sink[head] * L_LOG2E;
        L = 1.f;
    }
    for (int i0 = 0; i0 < n; i0 += AHEAD) {
        float2 ml[AHEAD];
        float4 o[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            ml[i] = make_float2(L_NEG_BIG, 0.f);
            o[i] = make_float4(0.f, 0.f, 0.f, 0.f);
            if (i0 + i < n) {
                const size_t slot = (size_t)p.merge_slots[b + i0 + i] * H + head;
                ml[i] = p.part_ml[slot];
                if (on) o[i] = *reinterpret_cast<const float4*>(p.part_o + slot * p.part_width + e);
            }
        }
        float top = M;
#pragma unroll
        for (int i = 0; i < AHEAD; i++) top = fmaxf(top, ml[i].x);
        const float keep = fast_exp2(M - top);
        M = top;
        L *= keep;
#pragma unroll
        for (int k = 0; k < 4; k++) acc[k] *= keep;
#pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            const float w = fast_exp2(ml[i].x - top);
            L = fmaf(w, ml[i].y, L);
            acc[0] = fmaf(w, o[i].x, acc[0]);
            acc[1] = fmaf(w, o[i].y, acc[1]);
            acc[2] = fmaf(w, o[i].z, acc[2]);
            acc[3] = fmaf(w, o[i].w, acc[3]);
        }
    }
    const float inv = L > 0.f ? 1.f / L : 0.f;
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + (size_t)blockIdx.x * p.kv_rank;
    if (p.kv_rank % 4 == 0) {
        if (e < p.kv_rank) *reinterpret_cast<uint2*>(out + e) = make_uint2(pack_bf16(acc[0] * inv, acc[1] * inv), pack_bf16(acc[2] * inv, acc[3] * inv));
    } else {
#pragma unroll
        for (int k = 0; k < 4; k++)
            if (e + k < p.kv_rank) out[e + k] = __float2bfloat16_rn(acc[k] * inv);
    }
}

constexpr int L_SMEM_LIMIT = 227 * 1024;
constexpr int L_CONTROL = (2 * L_MAX_UNITS + 7) * 8 + L_MAX_ROWS * 4 + 16;  // barriers, row factors, flags, TMEM address

template <int N> cudaError_t launch(const LatentParams& p, cudaStream_t stream) {
    const int tile_units = ((p.geo.gpr >> 3) + 1) / 2, fixed = layout_of<N>(p.geo.gpr, 0).end + L_CONTROL;
    // three tiles keep the copies ahead of the products; more would only keep other CTAs off the SM
    const int units = std::min({L_MAX_UNITS, 3 * tile_units, (L_SMEM_LIMIT - fixed) / L_UNIT});
    if (units < tile_units + 1) return cudaErrorInvalidValue;
    const int smem = units * L_UNIT + fixed;
    const int rows = p.path_off ? p.block_rows * p.n_heads : std::max(p.n_heads, p.item_rows);
    auto* span = latent_rows_kernel<N, true>;
    auto* items = latent_rows_kernel<N, false>;
    auto* k = p.path_off ? span : items;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributePreferredSharedMemoryCarveout, cudaSharedmemCarveoutMaxShared);
    if (e != cudaSuccess) return e;
    k<<<dim3(p.path_off ? p.n_blocks : p.n_items, (rows + N - 1) / N), L_THREADS, smem, stream>>>(p, units);
    return cudaGetLastError();
}

}  // namespace

bool latent_rows_serves(const Geometry& g) {
    return g.esize == 2 && g.chunk_size == L_TOK && g.swz && g.d_head <= 640 && g.d_value <= 512;
}

cudaError_t launch_latent_rows(const LatentParams& p, cudaStream_t stream) {
    const int rows = p.path_off ? p.block_rows * p.n_heads : std::max(p.n_heads, p.item_rows);
    cudaError_t e = rows <= 16 ? launch<16>(p, stream) : (rows <= 32 ? launch<32>(p, stream) : launch<64>(p, stream));
    if (e != cudaSuccess || p.path_off) return e;
    const int64_t pairs = (int64_t)p.n_rows * p.n_heads;
    if (pairs > 0x7fffffff) return cudaErrorInvalidValue;
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)pairs);
    cfg.blockDim = dim3(128);
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    return cudaLaunchKernelEx(&cfg, latent_merge_kernel, p);
}

}  // namespace ca
