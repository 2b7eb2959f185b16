// Attention over a latent cache on tensor cores (bf16, mma.sync): decode items of the planner's work list, and portions of
// prompts where expanding the latents into per-head keys and values (ca_latent_span.cu) does not pay.
//
// A token's pool row is key and value of every head at once, so the query heads of a token, and the tokens of a block, are
// rows of ONE product against the rows staged in shared memory: row r is head r % H of token r / H.
//   S = Q K^T   the eight warps share the tile: MT 16-row groups x 8 / MT runs of tokens
//   softmax     fp32, log2 units, online; the runs of a row meet in shared memory.  Every row has a window: positions from
//               its own minus (window - 1) on
//   O += P V    V is the leading part of the same staged rows; a warp owns d_value / 8 columns of every row.  The weights
//               enter as a sum of two bf16 numbers, which keeps 16 bits of them
// Tiles are half or whole chunks, copied verbatim (the pool's lines are the swizzled layout ldmatrix reads without
// conflicts) by 1-D TMA bulk copies into a ring.  Decode emits one partial per row and item, combined by the merge kernel of
// ca_attn_rows.cu; portions emit finished rows.  Every wait is bounded: when one runs out a status is recorded, the copies in
// flight are waited for (again with the limit) and the rows stay unwritten.
#include <algorithm>

#include "ca_kernels.h"
#include "ca_plan.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int L_THREADS = 256, L_WARPS = 8, L_CHUNK = 64, L_MAX_STAGES = 6;
constexpr float L_NEG_BIG = -1.0e30f, L_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ void sts32(uint32_t addr, uint32_t v) { asm volatile("st.shared.u32 [%0], %1;" ::"r"(addr), "r"(v) : "memory"); }

// tokens of a tile, and byte offset of granule g of line t in panels of `lines` 128-byte lines
template <int MT> __host__ __device__ constexpr int tile_tokens() { return MT == 4 ? 32 : 64; }
template <int LINES> __device__ __forceinline__ uint32_t staged(int t, int g) {
    return (g >> 3) * (LINES * 128) + t * 128 + (((g & 7) ^ (t & 7)) << 4);
}
// hi (part 0) and lo (part 1) weights: granule g of row r.  A row of 32 tokens holds both parts in one line.
template <int MT> __device__ __forceinline__ uint32_t weight_at(int part, int r, int g) {
    if (MT == 4) return r * 128 + (((g + 4 * part) ^ (r & 7)) << 4);
    return part * (16 * MT * 128) + r * 128 + ((g ^ (r & 7)) << 4);
}
template <int MT> constexpr int weight_bytes() { return MT == 4 ? 64 * 128 : 2 * 16 * MT * 128; }

template <int MT, int NV, bool SPAN>
__global__ void __launch_bounds__(L_THREADS) latent_rows_kernel(const LatentParams p, int stages) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int NT = tile_tokens<MT>(), ROWS = 16 * MT, TS = L_WARPS / MT, RUN = NT / TS, NB = RUN / 8;
    __shared__ float red[TS][ROWS], alpha_s[ROWS], m_s[ROWS];
    __shared__ __align__(8) uint64_t full[L_MAX_STAGES];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int H = p.n_heads, gpr = p.geo.gpr, panels = gpr >> 3;
    const int q_bytes = ROWS * gpr * 16, stage_bytes = NT * gpr * 16;
    const uint32_t q_base = smem_u32(smem), ring = q_base + q_bytes, w_base = ring + stages * stage_bytes;
    const uint32_t bars = smem_u32(full);

    // ---- the block of rows and its tokens: [start, end) relative to position `first` of list[0]
    int token0, n_rows, first, end, low, row_lo = 0, slot_base = 0;
    const int32_t* list;
    if (SPAN) {
        const int4 b = reinterpret_cast<const int4*>(p.blocks)[blockIdx.x];
        token0 = b.y;
        n_rows = (b.z - b.y) * H;
        first = 0;
        list = p.path_chunks + p.path_off[b.x];
        row_lo = (int)blockIdx.y * ROWS;
        if (row_lo >= n_rows) return;
        n_rows = min(ROWS, n_rows - row_lo);
        end = p.positions[token0 + (row_lo + n_rows - 1) / H] + 1;
        low = p.positions[token0 + row_lo / H];
    } else {
        const int* it = reinterpret_cast<const int*>(p.items) + 16 * blockIdx.x;
        const int n_tiles = it[0], flags = it[5], last = it[6];
        first = it[1];
        token0 = it[2];
        n_rows = it[3] * H;
        slot_base = it[4];
        list = it + 7;
        end = (n_tiles - 1) * L_CHUNK + min(L_CHUNK, last + ((flags & ITEM_FLAG_TAIL) ? p.delta_tokens : 0));
        low = p.positions[token0];
        for (int i = 1; i < it[3]; i++) low = min(low, p.positions[token0 + i]);
        row_lo = (int)blockIdx.y * ROWS;
        if (row_lo >= n_rows) return;
        n_rows = min(ROWS, n_rows - row_lo);
    }
    const int start = p.window > 0 ? max(0, low - p.window + 1 - first) / NT * NT : 0;
    const int n_tiles = end > start ? (end - start + NT - 1) / NT : 0;
    const int m_tiles = (n_rows + 15) >> 4;

    if (tid == 0) {
        for (int i = 0; i < stages; i++) mbar_init(bars + 8 * i, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    auto copy_tile = [&](int j) {  // one thread
        const int at = start + j * NT, lines = min(NT, end - at);
        const uint32_t dst = ring + (j % stages) * stage_bytes, bar = bars + 8 * (j % stages);
        int chunk = __ldg(list + at / L_CHUNK);
        if (chunk < 0 || chunk >= p.max_chunks) {
            atomicCAS(p.status, STATUS_OK, STATUS_BAD_WORK_LIST);
            chunk = 0;
        }
        const uint8_t* src = static_cast<const uint8_t*>(p.pool) + (size_t)chunk * (L_CHUNK * 16) * gpr + (at % L_CHUNK) * 128;
        mbar_arrive_expect_tx(bar, lines * gpr * 16);
        if (lines == L_CHUNK) {
            bulk_copy_g2s(dst, src, stage_bytes, bar);
        } else {
            for (int pn = 0; pn < panels; pn++) bulk_copy_g2s(dst + pn * (NT * 128), src + pn * (L_CHUNK * 128), lines * 128, bar);
        }
    };
    if (tid == 0)
        for (int j = 0; j < min(stages - 1, n_tiles); j++) copy_tile(j);

    // ---- queries: latent part as it comes, shared part turned by the row's position, zeros up to the pool's row
    {
        const bool whole = p.kv_rank % 8 == 0 && reinterpret_cast<uintptr_t>(p.q_lat) % 16 == 0;
        const __nv_bfloat16* q_lat = static_cast<const __nv_bfloat16*>(p.q_lat);
        const __nv_bfloat16* q_rot = static_cast<const __nv_bfloat16*>(p.q_rot);
        const int half = p.rot / 2;
        for (int i = tid; i < ROWS * gpr; i += L_THREADS) {
            const int r = i / gpr, g = i % gpr, rr = row_lo + r, token = token0 + rr / H, head = rr % H;
            uint4 v = make_uint4(0u, 0u, 0u, 0u);
            if (r < n_rows) {
                const __nv_bfloat16* src = q_lat + ((size_t)token * H + head) * p.kv_rank;
                if (whole && 8 * g < p.kv_rank) {
                    v = *reinterpret_cast<const uint4*>(src + 8 * g);
                } else if (8 * g < p.kv_rank + p.rot) {
                    const __nv_bfloat16* qr = q_rot + (size_t)token * p.q_rot_row + (size_t)head * p.q_rot_head;
                    float x[8];
#pragma unroll
                    for (int k = 0; k < 8; k++) {
                        const int e = 8 * g + k, d = e - p.kv_rank;
                        x[k] = 0.f;
                        if (d < 0) {
                            x[k] = __bfloat162float(src[e]);
                        } else if (d < p.rot) {
                            const int pair = d < half ? d : d - half;
                            float sn, cs;
                            fast_sincos((float)p.positions[token] * p.freq[pair], &sn, &cs);
                            const float a = __bfloat162float(qr[pair]), b = __bfloat162float(qr[pair + half]);
                            x[k] = d < half ? a * cs - b * sn : b * cs + a * sn;
                        }
                    }
                    v = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
                }
            }
            sts128(q_base + staged<ROWS>(r, g), (int)v.x, (int)v.y, (int)v.z, (int)v.w);
        }
    }

    // ---- roles: rows and tokens of the first product, columns of the second
    const int my_m = warp % MT, my_run = warp / MT;
    const bool busy = my_m < m_tiles;
    int lo[2], hi[2];  // positions a row sees, relative to `first`
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int r = my_m * 16 + (lane >> 2) + 8 * h;
        lo[h] = hi[h] = 0;
        if (r < n_rows) {
            const int pos = p.positions[token0 + (row_lo + r) / H] - first;
            hi[h] = min(pos + 1, end);
            lo[h] = p.window > 0 ? pos - p.window + 1 : 0;
        }
    }
    float o[MT][NV][4], m[2] = {L_NEG_BIG, L_NEG_BIG}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int i = 0; i < NV; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) o[a][i][k] = 0.f;
    const int mat = lane >> 3, r8 = lane & 7;
    __syncthreads();  // the queries are staged

    for (int j = 0; j < n_tiles; j++) {
        const uint32_t tile = ring + (j % stages) * stage_bytes;
        bool ok = mbar_wait_bounded(bars + 8 * (j % stages), (j / stages) & 1, p.wait_limit);
        ok = __all_sync(0xffffffffu, ok);
        const int at = start + j * NT, lines = min(NT, end - at);
        if (lines < NT) {
            // the lines behind the stored ones meet weights of zero and only have to be finite
            for (int i = tid; i < panels * (NT - lines) * 8; i += L_THREADS) {
                const int pn = i / ((NT - lines) * 8), q = i % ((NT - lines) * 8);
                sts128_zero(tile + pn * (NT * 128) + lines * 128 + q * 16);
            }
        }
        // ---- scores of 16 rows x RUN tokens
        float s[NB][4];
#pragma unroll
        for (int i = 0; i < NB; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) s[i][k] = 0.f;
        const int tb = my_run * RUN;
        if (busy && ok) {
            const int a_row = my_m * 16 + (lane & 15), a_g = lane >> 4;
            if (NB == 2) {
#pragma unroll 4
                for (int ks = 0; ks < gpr / 2; ks++) {
                    uint32_t a[4], b0, b1, b2, b3;
                    ldsm_x4(a[0], a[1], a[2], a[3], q_base + staged<ROWS>(a_row, 2 * ks + a_g));
                    ldsm_x4(b0, b1, b2, b3, tile + staged<NT>(tb + (mat >> 1) * 8 + r8, 2 * ks + (mat & 1)));
                    mma_bf16(s[0], a, b0, b1);
                    mma_bf16(s[NB - 1], a, b2, b3);
                }
            } else {
                float s2[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
                for (int ks = 0; ks < gpr / 2; ks += 2) {
                    uint32_t a[4], c[4], b0, b1, b2, b3;
                    ldsm_x4(a[0], a[1], a[2], a[3], q_base + staged<ROWS>(a_row, 2 * ks + a_g));
                    ldsm_x4(c[0], c[1], c[2], c[3], q_base + staged<ROWS>(a_row, 2 * ks + 2 + a_g));
                    ldsm_x4(b0, b1, b2, b3, tile + staged<NT>(tb + r8, 2 * ks + mat));
                    mma_bf16(s[0], a, b0, b1);
                    mma_bf16(s2, c, b2, b3);
                }
#pragma unroll
                for (int k = 0; k < 4; k++) s[0][k] += s2[k];
            }
        }
        const int col = at + tb + (lane & 3) * 2;  // of s[i][0], relative to `first`: + 8 i
        float mx[2] = {L_NEG_BIG, L_NEG_BIG};
#pragma unroll
        for (int i = 0; i < NB; i++)
#pragma unroll
            for (int k = 0; k < 4; k++) {
                const int c = col + 8 * i + (k & 1);
                s[i][k] = c >= lo[k >> 1] && c < hi[k >> 1] ? s[i][k] * p.scale_log2 : -INFINITY;
                mx[k >> 1] = fmaxf(mx[k >> 1], s[i][k]);
            }
#pragma unroll
        for (int h = 0; h < 2; h++) {
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
            mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
            if ((lane & 3) == 0) red[my_run][my_m * 16 + (lane >> 2) + 8 * h] = mx[h];
        }
        if (!__syncthreads_and(ok)) {
            if (tid == 0) {
                atomicCAS(p.status, STATUS_OK, STATUS_FULL_WAIT_TIMEOUT);
                for (int f = j; f < min(n_tiles, j + stages - 1); f++)
                    mbar_wait_bounded(bars + 8 * (f % stages), (f / stages) & 1, p.wait_limit);
            }
            return;
        }
        // every warp is past tile j - 1: its slot takes tile j + stages - 1
        if (tid == 0 && j + stages - 1 < n_tiles) copy_tile(j + stages - 1);
        if (busy) {
            float alpha[2];
#pragma unroll
            for (int h = 0; h < 2; h++) {
                const int r = my_m * 16 + (lane >> 2) + 8 * h;
                float mn = m[h];
#pragma unroll
                for (int t = 0; t < TS; t++) mn = fmaxf(mn, red[t][r]);
                alpha[h] = fast_exp2(m[h] - mn);
                m[h] = mn;
                if (my_run == 0 && (lane & 3) == 0) alpha_s[r] = alpha[h];
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < NB; i++) {
                    const float a = fast_exp2(s[i][2 * h] - mn), b = fast_exp2(s[i][2 * h + 1] - mn);
                    sum += a + b;
                    const uint32_t hw = pack_bf16(a, b);
                    const uint32_t lw = pack_bf16(a - __uint_as_float(hw << 16), b - __uint_as_float(hw & 0xffff0000u));
                    const int t = tb + 8 * i + (lane & 3) * 2;
                    sts32(w_base + weight_at<MT>(0, r, t >> 3) + (t & 7) * 2, hw);
                    sts32(w_base + weight_at<MT>(1, r, t >> 3) + (t & 7) * 2, lw);
                }
                l[h] = l[h] * alpha[h] + sum;  // this lane's tokens only
            }
        }
        __syncthreads();
        // ---- O += P V over this warp's columns
        const int c0 = warp * (8 * NV);
        if (c0 < p.geo.d_value) {
#pragma unroll
            for (int a = 0; a < MT; a++)
                if (a < m_tiles) {
                    const float x = alpha_s[a * 16 + (lane >> 2)], y = alpha_s[a * 16 + (lane >> 2) + 8];
                    if (__any_sync(0xffffffffu, x != 1.f || y != 1.f)) {
#pragma unroll
                        for (int i = 0; i < NV; i++) {
                            o[a][i][0] *= x;
                            o[a][i][1] *= x;
                            o[a][i][2] *= y;
                            o[a][i][3] *= y;
                        }
                    }
                }
#pragma unroll
            for (int kk = 0; kk < NT / 16; kk++) {
                uint32_t b[NV][2];
#pragma unroll
                for (int i = 0; i < NV; i += 2) {
                    // columns past d_value (NV rounded up) are neither read nor stored
                    const int c = c0 + 8 * i < p.geo.d_value ? c0 + 8 * i : c0;
                    ldsm_x4_trans(b[i][0], b[i][1], b[i + 1][0], b[i + 1][1],
                                  tile + staged<NT>(16 * kk + (mat & 1) * 8 + r8, c / 8 + (mat >> 1)));
                }
#pragma unroll
                for (int a = 0; a < MT; a++)
                    if (a < m_tiles) {
                        uint32_t hw[4], lw[4];
                        const int r = a * 16 + (lane & 15), g = 2 * kk + (lane >> 4);
                        ldsm_x4(hw[0], hw[1], hw[2], hw[3], w_base + weight_at<MT>(0, r, g));
                        ldsm_x4(lw[0], lw[1], lw[2], lw[3], w_base + weight_at<MT>(1, r, g));
#pragma unroll
                        for (int i = 0; i < NV; i++) {
                            mma_bf16(o[a][i], hw, b[i][0], b[i][1]);
                            mma_bf16(o[a][i], lw, b[i][0], b[i][1]);
                        }
                    }
            }
        }
    }

    // ---- sums of the runs, then every warp stores its columns
    __syncthreads();
#pragma unroll
    for (int h = 0; h < 2; h++) {
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
        l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
        const int r = my_m * 16 + (lane >> 2) + 8 * h;
        if ((lane & 3) == 0) {
            red[my_run][r] = l[h];
            if (my_run == 0) m_s[r] = m[h];
        }
    }
    __syncthreads();
    const int c0 = warp * (8 * NV);
#pragma unroll
    for (int a = 0; a < MT; a++)
#pragma unroll
        for (int h = 0; h < 2; h++) {
            const int r = a * 16 + (lane >> 2) + 8 * h;
            if (r >= n_rows) continue;
            float M = m_s[r], L = 0.f;
#pragma unroll
            for (int t = 0; t < TS; t++) L += red[t][r];
            const int rr = row_lo + r, token = token0 + rr / H, head = rr % H;
            if (SPAN) {
                float f = 1.f;
                if (p.sink) {
                    const float sk = p.sink[head] * L_LOG2E, top = fmaxf(M, sk);
                    f = fast_exp2(M - top);
                    L = L * f + fast_exp2(sk - top);
                }
                f = L > 0.f ? f / L : 0.f;
                __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + ((size_t)token * H + head) * p.kv_rank;
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    const int c = c0 + 8 * i + (lane & 3) * 2;
                    const float x = o[a][i][2 * h] * f, y = o[a][i][2 * h + 1] * f;
                    if (p.kv_rank % 2 == 0) {
                        if (c < p.kv_rank) *reinterpret_cast<uint32_t*>(out + c) = pack_bf16(x, y);
                    } else {
                        if (c < p.kv_rank) out[c] = __float2bfloat16_rn(x);
                        if (c + 1 < p.kv_rank) out[c + 1] = __float2bfloat16_rn(y);
                    }
                }
            } else {
                const size_t slot = (size_t)slot_base * H + (size_t)(rr / H) * H + head;
                if (warp == 0 && (lane & 3) == 0) p.part_ml[slot] = make_float2(M, L);
                float* dst = p.part_o + slot * p.part_width;
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    const int c = c0 + 8 * i + (lane & 3) * 2;
                    if (c < p.part_width) *reinterpret_cast<float2*>(dst + c) = make_float2(o[a][i][2 * h], o[a][i][2 * h + 1]);
                }
            }
        }
}

constexpr int L_SMEM_LIMIT = 227 * 1024 - 2048;  // static shared memory and alignment taken off

template <int MT, int NV> cudaError_t launch(const LatentParams& p, cudaStream_t stream) {
    const int q_bytes = 16 * MT * p.geo.gpr * 16, stage = tile_tokens<MT>() * p.geo.gpr * 16, weights = weight_bytes<MT>();
    const int room = (L_SMEM_LIMIT - q_bytes - weights) / stage;
    if (room < 2) return cudaErrorInvalidValue;
    const int stages = std::min(room, L_MAX_STAGES), smem = q_bytes + stages * stage + weights;
    const unsigned subs = (unsigned)((p.path_off ? p.block_rows * p.n_heads : std::max(p.n_heads, p.item_rows)) + 16 * MT - 1) / (16 * MT);
    if (p.path_off) {
        auto* k = latent_rows_kernel<MT, NV, true>;
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        k<<<dim3(p.n_blocks, subs), L_THREADS, smem, stream>>>(p, stages);
    } else {
        auto* k = latent_rows_kernel<MT, NV, false>;
        cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
        if (e != cudaSuccess) return e;
        k<<<dim3(p.n_items, subs), L_THREADS, smem, stream>>>(p, stages);
    }
    return cudaGetLastError();
}

template <int MT> cudaError_t by_width(const LatentParams& p, cudaStream_t stream) {
    if (p.geo.d_value <= 128) return launch<MT, 2>(p, stream);
    if (p.geo.d_value <= 256) return launch<MT, 4>(p, stream);
    return launch<MT, 8>(p, stream);
}

}  // namespace

bool latent_rows_serves(const Geometry& g) {
    return g.esize == 2 && g.chunk_size == L_CHUNK && g.swz && g.d_head <= 640 && g.d_value <= 512;
}

cudaError_t launch_latent_rows(const LatentParams& p, cudaStream_t stream) {
    const int rows = p.path_off ? std::min(64, p.block_rows * p.n_heads) : std::max(p.n_heads, p.item_rows);
    cudaError_t e = rows <= 16 ? by_width<1>(p, stream) : (rows <= 32 ? by_width<2>(p, stream) : by_width<4>(p, stream));
    if (e != cudaSuccess || p.path_off) return e;
    RowsParams r{};
    r.geo = p.geo;
    r.group = p.n_heads;
    r.out = p.out;
    r.out_width = p.kv_rank;
    r.n_rows = p.n_rows;
    r.sink_scores = p.sink;
    r.part_o = p.part_o;
    r.part_ml = p.part_ml;
    r.part_width = p.part_width;
    r.merge_off = p.merge_off;
    r.merge_slots = p.merge_slots;
    return launch_rows_merge(r, stream);
}

}  // namespace ca
