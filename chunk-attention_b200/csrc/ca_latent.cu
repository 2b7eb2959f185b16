// Latent caches: one row per token for all heads, a normalised latent vector followed by a rotated key part that the heads
// share.  Here are the kernel that fills them from a batch's projections, the attention kernel for any geometry and type
// (the float32 mode, and bf16 where ca_latent_rows.cu does not apply), and the gather that lays the rows a step of
// portions reads out densely.
#include <algorithm>

#include "ca_kernels.h"
#include "ca_types.cuh"

namespace ca {
namespace {

// ---- projections -> query latent and pool row --------------------------------------------------------------------
// One CTA per token.  V elements per access (whole granules), or 1.  Everything the token needs is requested before the
// reduction; what a thread does not keep in registers (longer rows) is read again.
constexpr int LS_THREADS = 128, LS_KEEP_Q = 2;

__device__ __forceinline__ float2 block_sum2(float a, float b) {
    __shared__ float2 sums[LS_THREADS / 32];
    a = warp_sum(a);
    b = warp_sum(b);
    if ((threadIdx.x & 31) == 0) sums[threadIdx.x >> 5] = make_float2(a, b);
    __syncthreads();
    float2 s = make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < LS_THREADS / 32; i++) {
        s.x += sums[i].x;
        s.y += sums[i].y;
    }
    return s;
}

template <typename T, int V>
__global__ void __launch_bounds__(LS_THREADS) latent_store_kernel(const LatentStoreParams p) {
    using P = Pack<T, V>;
    using W = Pack<float, V>;
    const int t = blockIdx.x, tid = threadIdx.x, c0 = tid * V, step = LS_THREADS * V;
    const T* row = static_cast<const T*>(p.in) + (size_t)t * p.row_stride;
    const T* kv = row + p.q_rank;
    const T* r = kv + p.kv_rank;
    auto squares = [](const P& a) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < V; i++) {
            const float x = to_f32(a.v[i]);
            s = fmaf(x, x, s);
        }
        return s;
    };
    P q_keep[LS_KEEP_Q], kv_keep{};
#pragma unroll
    for (int k = 0; k < LS_KEEP_Q; k++) {
        q_keep[k] = P{};
        if (c0 + k * step < p.q_rank) q_keep[k] = *reinterpret_cast<const P*>(row + c0 + k * step);
    }
    if (c0 < p.kv_rank) kv_keep = *reinterpret_cast<const P*>(kv + c0);
    int chunk, slot;
    if (p.tok_slot) {
        const int s = p.tok_slot[t];
        chunk = s < 0 ? -1 : s / p.geo.chunk_size;
        slot = s - chunk * p.geo.chunk_size;
    } else {
        chunk = p.tail_chunk[t];
        slot = p.tail_tokens[t] + p.delta_tokens;
        if (slot >= p.geo.chunk_size) chunk = -1;  // rejected on the host; never write past the tile
    }
    const int half = p.rot / 2;
    float rot_u = 0.f, rot_v = 0.f, sn = 0.f, cs = 0.f;
    if (tid < half) {
        turn_for<T>((float)p.positions[t], p.freq[tid], p.freq[half + tid], &sn, &cs);
        rot_u = to_f32(r[tid]);
        rot_v = to_f32(r[tid + half]);
    }
    float sq = 0.f, skv = squares(kv_keep);
#pragma unroll
    for (int k = 0; k < LS_KEEP_Q; k++) sq += squares(q_keep[k]);
    for (int c = c0 + LS_KEEP_Q * step; c < p.q_rank; c += step) sq += squares(*reinterpret_cast<const P*>(row + c));
    for (int c = c0 + step; c < p.kv_rank; c += step) skv += squares(*reinterpret_cast<const P*>(kv + c));
    const float2 ss = block_sum2(sq, skv);

    auto scaled = [](const P& a, float inv, const float* w) {
        const W ww = *reinterpret_cast<const W*>(w);
        P o;
#pragma unroll
        for (int i = 0; i < V; i++) o.v[i] = from_f32<T>(to_f32(a.v[i]) * inv * ww.v[i]);
        return o;
    };
    if (p.q_rank > 0) {
        const float inv = 1.f / sqrtf(ss.x / p.q_rank + p.eps);
        T* out = static_cast<T*>(p.q_out) + (size_t)t * p.q_rank;
#pragma unroll
        for (int k = 0; k < LS_KEEP_Q; k++) {
            const int c = c0 + k * step;
            if (c < p.q_rank) *reinterpret_cast<P*>(out + c) = scaled(q_keep[k], inv, p.q_norm + c);
        }
        for (int c = c0 + LS_KEEP_Q * step; c < p.q_rank; c += step)
            *reinterpret_cast<P*>(out + c) = scaled(*reinterpret_cast<const P*>(row + c), inv, p.q_norm + c);
    }
    if (chunk < 0) return;
    T* tile = static_cast<T*>(p.pool) + tile_base_elems(p.geo, chunk, 0, 0);
    const float inv = 1.f / sqrtf(ss.y / p.kv_rank + p.eps);
    for (int c = c0; c < p.kv_rank; c += step)
        *reinterpret_cast<P*>(tile + tile_elem_offset(p.geo, slot, c)) = scaled(c == c0 ? kv_keep : *reinterpret_cast<const P*>(kv + c), inv, p.kv_norm + c);
    for (int i = tid; i < half; i += LS_THREADS) {
        if (i != tid) {
            turn_for<T>((float)p.positions[t], p.freq[i], p.freq[half + i], &sn, &cs);
            rot_u = to_f32(r[i]);
            rot_v = to_f32(r[i + half]);
        }
        tile[tile_elem_offset(p.geo, slot, p.kv_rank + i)] = from_f32<T>(rot_u * cs - rot_v * sn);
        tile[tile_elem_offset(p.geo, slot, p.kv_rank + half + i)] = from_f32<T>(rot_v * cs + rot_u * sn);
    }
    for (int c = p.kv_rank + p.rot + tid; c < p.geo.d_head; c += LS_THREADS) tile[tile_elem_offset(p.geo, slot, c)] = from_f32<T>(0.f);
}

template <typename T> void run_latent_store(const LatentStoreParams& p, cudaStream_t stream) {
    constexpr int V = 16 / sizeof(T);
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    auto aligned32 = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 32 == 0; };
    if (p.q_rank % V == 0 && p.kv_rank % V == 0 && p.row_stride % V == 0 && aligned(p.in) && aligned(p.q_out) && aligned32(p.q_norm) &&
        aligned32(p.kv_norm))
        latent_store_kernel<T, V><<<p.n_tokens, LS_THREADS, 0, stream>>>(p);
    else
        latent_store_kernel<T, 1><<<p.n_tokens, LS_THREADS, 0, stream>>>(p);
}

// ---- attention, any geometry -----------------------------------------------------------------------------------------
// One CTA of four warps per (row, head): the positions of the row's window are cut into blocks of 32 tokens which the warps
// take in turn; lane j scores token j against the query in shared memory (its last part rotated there by the row's
// position), then every lane walks the block's tokens over the granules of the output row it owns.
constexpr int LG_WARPS = 4, LG_MAX_V = 1024, LG_MAX_K = 1152;

template <typename T>
__global__ void __launch_bounds__(LG_WARPS * 32) latent_generic_kernel(const LatentParams p) {
    constexpr int EPG = 16 / sizeof(T), OWN = LG_MAX_V / EPG / 32;  // granules a lane may own
    __shared__ float q_s[LG_MAX_K];
    __shared__ float part[LG_WARPS][LG_MAX_V];
    __shared__ float ml[LG_WARPS][2];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int H = p.n_heads, row = blockIdx.x / H, head = blockIdx.x % H;
    const int kv_rank = p.kv_rank, rot = p.rot, C = p.geo.chunk_size;
    const int pos = p.positions[row];
    {
        const T* q = static_cast<const T*>(p.q_lat) + ((size_t)row * H + head) * kv_rank;
        const T* qr = static_cast<const T*>(p.q_rot) + (size_t)row * p.q_rot_row + (size_t)head * p.q_rot_head;
        for (int e = threadIdx.x; e < p.geo.d_head; e += blockDim.x)
            if (e < kv_rank || e >= kv_rank + rot) q_s[e] = e < kv_rank ? to_f32(q[e]) * p.scale : 0.f;
        const int half = rot / 2;
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            float sn, cs;
            turn_for<T>((float)pos, p.freq[i], p.freq[half + i], &sn, &cs);
            const float u = to_f32(qr[i]), v = to_f32(qr[i + half]);
            // rounded as the tensor-core kernels' operands are
            q_s[kv_rank + i] = to_f32(from_f32<T>(u * cs - v * sn)) * p.scale;
            q_s[kv_rank + half + i] = to_f32(from_f32<T>(v * cs + u * sn)) * p.scale;
        }
    }
    __syncthreads();
    float o[OWN][EPG];
#pragma unroll
    for (int i = 0; i < OWN; i++)
#pragma unroll
        for (int k = 0; k < EPG; k++) o[i][k] = 0.f;
    float m = -INFINITY, l = 0.f;
    const int32_t* list = p.path_chunks + p.path_off[p.row_entry[row]];
    const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    const int v_gr = (kv_rank + EPG - 1) / EPG;
    const T* pool = static_cast<const T*>(p.pool);
    for (int t0 = lo + warp * 32; t0 <= pos; t0 += LG_WARPS * 32) {
        const int nv = min(32, pos + 1 - t0), t = t0 + lane;
        float sc = -INFINITY;
        if (lane < nv) {
            const T* tile = pool + tile_base_elems(p.geo, list[t / C], 0, 0);
            float acc = 0.f;
            for (int g = 0; g < p.geo.gpr; g++) {
                float kf[EPG];
                Granule<T>::load(tile + tile_granule_index(p.geo, t % C, g) * EPG, kf);
#pragma unroll
                for (int k = 0; k < EPG; k++) acc = fmaf(q_s[g * EPG + k], kf[k], acc);
            }
            sc = acc;
        }
        const float mn = fmaxf(m, warp_max(sc));
        const float alpha = expf(m - mn);
        const float pj = lane < nv ? expf(sc - mn) : 0.f;
        l = l * alpha + warp_sum(pj);
        m = mn;
#pragma unroll
        for (int i = 0; i < OWN; i++)
#pragma unroll
            for (int k = 0; k < EPG; k++) o[i][k] *= alpha;
        for (int j = 0; j < nv; j++) {
            const float pw = __shfl_sync(0xffffffffu, pj, j);
            const T* tile = pool + tile_base_elems(p.geo, list[(t0 + j) / C], 0, 0);
#pragma unroll
            for (int i = 0; i < OWN; i++) {
                const int g = lane + 32 * i;
                if (g < v_gr) {
                    float vf[EPG];
                    Granule<T>::load(tile + tile_granule_index(p.geo, (t0 + j) % C, g) * EPG, vf);
#pragma unroll
                    for (int k = 0; k < EPG; k++) o[i][k] = fmaf(pw, vf[k], o[i][k]);
                }
            }
        }
    }
    if (lane == 0) {
        ml[warp][0] = m;
        ml[warp][1] = l;
    }
#pragma unroll
    for (int i = 0; i < OWN; i++) {
        const int g = lane + 32 * i;
        if (g < v_gr) {
#pragma unroll
            for (int k = 0; k < EPG; k++) part[warp][g * EPG + k] = o[i][k];
        }
    }
    __syncthreads();
    const float sink = p.sink ? p.sink[head] : -INFINITY;
    float mm = sink;
#pragma unroll
    for (int w = 0; w < LG_WARPS; w++) mm = fmaxf(mm, ml[w][0]);
    float wgt[LG_WARPS], ll = p.sink ? expf(sink - mm) : 0.f;
#pragma unroll
    for (int w = 0; w < LG_WARPS; w++) {
        wgt[w] = ml[w][1] > 0.f ? expf(ml[w][0] - mm) : 0.f;
        ll = fmaf(wgt[w], ml[w][1], ll);
    }
    const float inv = ll > 0.f ? 1.f / ll : 0.f;
    T* out = static_cast<T*>(p.out) + ((size_t)row * H + head) * kv_rank;
    for (int e = threadIdx.x; e < kv_rank; e += blockDim.x) {
        float acc = 0.f;
#pragma unroll
        for (int w = 0; w < LG_WARPS; w++) acc = fmaf(wgt[w], part[w][e], acc);
        out[e] = from_f32<T>(acc * inv);
    }
}

// ---- pool rows of a step's windows, laid out densely --------------------------------------------------------------------
// One warp per workspace row.
template <typename T>
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherParams p) {
    constexpr int EPG = 16 / sizeof(T);
    const int row = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= p.n_rows) return;
    const int C = p.geo.chunk_size, src = p.src_row[row], at = src % C;
    int chunk = src / C;
    if (src < 0 || chunk >= p.max_chunks) {
        if (lane == 0) atomicCAS(p.status, STATUS_OK, STATUS_BAD_WORK_LIST);
        chunk = 0;
    }
    const T* tile = static_cast<const T*>(p.pool) + tile_base_elems(p.geo, chunk, 0, 0);
    T* lat = static_cast<T*>(p.lat) + (size_t)row * p.kv_rank;
    T* rot = static_cast<T*>(p.rot) + (size_t)row * p.rot_stride;
    if (p.kv_rank % EPG == 0) {
        const int n = p.kv_rank / EPG;
        using P = Pack<T, EPG>;
        for (int g = lane; g < n; g += 32)
            reinterpret_cast<P*>(lat)[g] = *reinterpret_cast<const P*>(tile + tile_granule_index(p.geo, at, g) * EPG);
        for (int g = lane; g < p.rot_stride / EPG; g += 32) {  // what lies behind the rotated elements is zero in the pool, too
            P a{};
            if (n + g < p.geo.gpr) a = *reinterpret_cast<const P*>(tile + tile_granule_index(p.geo, at, n + g) * EPG);
            reinterpret_cast<P*>(rot)[g] = a;
        }
    } else {
        for (int c = lane; c < p.kv_rank; c += 32) lat[c] = tile[tile_elem_offset(p.geo, at, c)];
        for (int c = lane; c < p.rot_stride; c += 32)
            rot[c] = c < p.rot_dims ? tile[tile_elem_offset(p.geo, at, p.kv_rank + c)] : from_f32<T>(0.f);
    }
}

}  // namespace

cudaError_t launch_latent_store(const LatentStoreParams& p, int dtype, cudaStream_t stream) {
    if (p.n_tokens <= 0) return cudaSuccess;
    if (dtype == 2) run_latent_store<__nv_bfloat16>(p, stream);
    else if (dtype == 1) run_latent_store<float>(p, stream);
    else return cudaErrorInvalidValue;
    return cudaGetLastError();
}

cudaError_t launch_latent_generic(const LatentParams& p, int dtype, cudaStream_t stream) {
    const int64_t pairs = (int64_t)p.n_rows * p.n_heads;
    if (pairs <= 0) return cudaSuccess;
    if (pairs > 0x7fffffff || p.kv_rank > LG_MAX_V || p.geo.d_head > LG_MAX_K || p.geo.epg < 2) return cudaErrorInvalidValue;
    if (dtype == 2) latent_generic_kernel<__nv_bfloat16><<<(unsigned)pairs, LG_WARPS * 32, 0, stream>>>(p);
    else if (dtype == 1) latent_generic_kernel<float><<<(unsigned)pairs, LG_WARPS * 32, 0, stream>>>(p);
    else return cudaErrorInvalidValue;
    return cudaGetLastError();
}

cudaError_t launch_latent_gather(const LatentGatherParams& p, int dtype, cudaStream_t stream) {
    if (p.n_rows <= 0) return cudaSuccess;
    const unsigned grid = (unsigned)((p.n_rows + 7) / 8);
    if (dtype == 2) latent_gather_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(p);
    else if (dtype == 1) latent_gather_kernel<float><<<grid, 256, 0, stream>>>(p);
    else return cudaErrorInvalidValue;
    return cudaGetLastError();
}

}  // namespace ca
