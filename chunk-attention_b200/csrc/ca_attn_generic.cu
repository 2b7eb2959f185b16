// Sequence-first-only attention for any geometry (fp16, bf16 or fp32, d_head <= 256, any chunk
// size), fp32 arithmetic with accurate expf.  It serves the geometries the tensor-core/TMA kernels
// do not (the reference's CPU tests use fp32 with d_head 4..128 and chunk sizes 2..1024,
// tests/test_chunk_attn_cpu.py:24-385), `partition = 2` requests (the reference's
// sequence-first-only mode, cpp/chunk_attn/kernel_cpu_mkl.cpp:122-242), and is the in-library
// cross-check of the fast path.
//
// One CTA of 4 warps per (row, head).  The row's root-to-leaf chunk path is cut into blocks of 32
// tokens which the warps take in turn.  For a block, lane j computes the score of token j (a dot
// product along the token's K row, read in 16-byte granules against the query held in shared
// memory), the block's maximum and sum come from warp shuffles, and the P.V update walks the 32
// tokens with each lane owning one or two 16-byte granules of the output row (coalesced V reads).
// The four warps' (max, sum, O) are combined through shared memory at the end.  Rows whose length
// is not a whole number of 16-byte granules (odd d_head), or an unaligned pool, take an element-wise
// variant of the same walk.
//
// A row is one query token: the last token of a sequence (decode), or token t of a batch of portions
// (prefill), which then sees the positions up to its own.  Grouped heads, values of another width
// than the keys, a unit term in the softmax denominator and values cached rotated by their position
// (the output row is turned back) are parameters of the walk.
#include "ca_kernels.h"
#include "ca_types.cuh"

namespace ca {
namespace {

constexpr int GEN_WARPS = 4;
constexpr int GEN_MAX_D = 256;

// VEC: rows are whole 16-byte granules (geo.epg > 1); a lane owns granules lane and lane + 32 of the
// output row.  Otherwise a lane owns elements lane + 32 i.
template <typename T, bool VEC>
__global__ void __launch_bounds__(GEN_WARPS * 32) attn_seq_generic_kernel(const GenericParams p) {
    constexpr int EPG = Granule<T>::N;
    constexpr int OWN = VEC ? 2 * EPG : GEN_MAX_D / 32;  // output elements a lane may own
    __shared__ float q_s[GEN_MAX_D];
    __shared__ float part[GEN_WARPS][GEN_MAX_D + 2];

    const int pair = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n_q_heads = p.geo.n_heads * p.group;
    const int row = pair / n_q_heads;
    const int qh = pair - row * n_q_heads;
    const int h = qh / p.group;  // key/value head
    const int d = p.geo.d_head, dv = p.geo.d_value;
    const int gpr = p.geo.gpr, v_gpr = p.geo.v_gpr;
    const Geometry v_side = tile_side(p.geo, 1);
    const int s = p.row_entry ? p.row_entry[row] : row;  // whose path the row walks
    const int limit = p.row_entry ? p.positions[row] + 1 : 0x7fffffff;  // tokens of it the row sees
    const T* pool = reinterpret_cast<const T*>(p.pool);
    {
        const T* q = reinterpret_cast<const T*>(p.q) + (size_t)pair * d;
        for (int e = threadIdx.x; e < d; e += blockDim.x) q_s[e] = to_f32(q[e]) * p.scale;
    }
    __syncthreads();

    float o[OWN];
#pragma unroll
    for (int i = 0; i < OWN; i++) o[i] = 0.f;
    float m = -INFINITY, l = 0.f;

    const int pb = p.path_off[s], pe = p.path_off[s + 1];
    int turn = 0;  // blocks are dealt to the warps round-robin
    int first = 0; // position of the chunk's first token
    for (int pi = pb; pi < pe && first < limit; pi++) {
        int nt = p.path_tokens ? p.path_tokens[pi] : p.geo.chunk_size;
        if (pi == pe - 1 && p.path_tokens) nt = min(nt + p.delta_tokens, p.geo.chunk_size);  // the row's tail
        const int before = first;
        first += nt;
        nt = min(nt, limit - before);
        const T* kt = pool + tile_base_elems(p.geo, p.path_chunks[pi], h, 0);
        const T* vt = kt + p.geo.tile_elems;
        for (int t0 = 0; t0 < nt; t0 += 32, turn++) {
            if ((turn & (GEN_WARPS - 1)) != warp) continue;
            const int nv = min(32, nt - t0);
            const int t = t0 + lane;
            // ---- scores: lane j <-> token t0 + j
            float sc = -INFINITY;
            if (lane < nv) {
                float acc = 0.f;
                if (VEC) {
                    for (int g = 0; g < gpr; g++) {
                        float kf[EPG];
                        Granule<T>::load(kt + tile_granule_index(p.geo, t, g) * EPG, kf);
#pragma unroll
                        for (int k = 0; k < EPG; k++) acc = fmaf(q_s[g * EPG + k], kf[k], acc);
                    }
                } else {
                    for (int e = 0; e < d; e++) acc = fmaf(q_s[e], to_f32(kt[tile_elem_offset(p.geo, t, e)]), acc);
                }
                sc = acc;
            }
            // ---- online softmax over the block
            const float mn = fmaxf(m, warp_max(sc));
            const float alpha = expf(m - mn);  // exp(-inf) = 0 before the first token
            const float pj = lane < nv ? expf(sc - mn) : 0.f;
            l = l * alpha + warp_sum(pj);
            m = mn;
#pragma unroll
            for (int i = 0; i < OWN; i++) o[i] *= alpha;
            // ---- O += P V: every lane walks the block's tokens over the elements it owns
            for (int j = 0; j < nv; j++) {
                const float pw = __shfl_sync(0xffffffffu, pj, j);
                const int tj = t0 + j;
                if (VEC) {
#pragma unroll
                    for (int gi = 0; gi < 2; gi++) {
                        const int g = lane + 32 * gi;
                        if (g < v_gpr) {
                            float vf[EPG];
                            Granule<T>::load(vt + tile_granule_index(v_side, tj, g) * EPG, vf);
#pragma unroll
                            for (int k = 0; k < EPG; k++) o[gi * EPG + k] = fmaf(pw, vf[k], o[gi * EPG + k]);
                        }
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < OWN; i++) {
                        const int e = lane + 32 * i;
                        if (e < dv) o[i] = fmaf(pw, to_f32(vt[tile_elem_offset(v_side, tj, e)]), o[i]);
                    }
                }
            }
        }
    }

    // ---- combine the warps
    if (lane == 0) {
        part[warp][GEN_MAX_D] = m;
        part[warp][GEN_MAX_D + 1] = l;
    }
    if (VEC) {
#pragma unroll
        for (int gi = 0; gi < 2; gi++) {
            const int g = lane + 32 * gi;
            if (g < v_gpr) {
#pragma unroll
                for (int k = 0; k < EPG; k++) part[warp][g * EPG + k] = o[gi * EPG + k];
            }
        }
    } else {
#pragma unroll
        for (int i = 0; i < OWN; i++) {
            const int e = lane + 32 * i;
            if (e < dv) part[warp][e] = o[i];
        }
    }
    __syncthreads();
    float mm = p.sink ? 0.f : -INFINITY;  // the sink is a score of 0 without a value
#pragma unroll
    for (int w = 0; w < GEN_WARPS; w++) mm = fmaxf(mm, part[w][GEN_MAX_D]);
    float wgt[GEN_WARPS];
    float ll = p.sink ? expf(-mm) : 0.f;
#pragma unroll
    for (int w = 0; w < GEN_WARPS; w++) {
        // a warp that saw no token has max -inf and sum 0: it contributes nothing
        wgt[w] = part[w][GEN_MAX_D + 1] > 0.f ? expf(part[w][GEN_MAX_D] - mm) : 0.f;
        ll = fmaf(wgt[w], part[w][GEN_MAX_D + 1], ll);
    }
    const float inv = ll > 0.f ? 1.f / ll : 0.f;  // a row with no token yields zeros
    const int width = p.out_width;  // stored elements of a value row, without padding
    T* out = reinterpret_cast<T*>(p.out) + (size_t)pair * width;
    auto value = [&](int e) {
        float acc = 0.f;
#pragma unroll
        for (int w = 0; w < GEN_WARPS; w++) acc = fmaf(wgt[w], part[w][e], acc);
        return acc * inv;
    };
    if (!p.value_freq) {
        for (int e = threadIdx.x; e < width; e += blockDim.x) out[e] = from_f32<T>(value(e));
        return;
    }
    // values were cached turned by their own position: turn the sum back by the row's
    const float pos = (float)p.positions[row];
    for (int i = threadIdx.x; 2 * i < width; i += blockDim.x) {
        const float a = value(2 * i), b = 2 * i + 1 < width ? value(2 * i + 1) : 0.f;
        float sn, cs;
        sincosf(pos * p.value_freq[i], &sn, &cs);
        out[2 * i] = from_f32<T>(a * cs + b * sn);
        if (2 * i + 1 < width) out[2 * i + 1] = from_f32<T>(b * cs - a * sn);
    }
}

}  // namespace

cudaError_t launch_attn_seq_generic(const GenericParams& p, int dtype, cudaStream_t stream) {
    const int64_t pairs = (int64_t)p.n_rows * p.geo.n_heads * p.group;
    if (pairs <= 0) return cudaSuccess;
    if (p.geo.d_head > GEN_MAX_D || p.geo.d_value > GEN_MAX_D || pairs > 0x7fffffff) return cudaErrorInvalidValue;
    // 16-byte granule reads need the pool base aligned (rows and tiles then are, too)
    const bool vec = p.geo.epg > 1 && reinterpret_cast<uintptr_t>(p.pool) % 16 == 0;
    if (dtype == 2) {
        if (vec) attn_seq_generic_kernel<__nv_bfloat16, true><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
        else attn_seq_generic_kernel<__nv_bfloat16, false><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
    } else if (dtype == 0) {
        if (vec) attn_seq_generic_kernel<__half, true><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
        else attn_seq_generic_kernel<__half, false><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
    } else {
        if (vec) attn_seq_generic_kernel<float, true><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
        else attn_seq_generic_kernel<float, false><<<(unsigned)pairs, GEN_WARPS * 32, 0, stream>>>(p);
    }
    return cudaGetLastError();
}

}  // namespace ca
