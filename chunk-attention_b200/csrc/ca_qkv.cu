// From the projections of a batch of tokens to attention operands, in one kernel: per-head RMS norm of q and k,
// rotation of q and k (interleaved pairs, a leading part of each head), rotation of v by its position, and the
// store - q to a dense buffer, k and v straight into the token's row of the chunk pool.  A decode step writes row
// s of the batch into the next free row of sequence s's tail chunk; a portion of a prompt names the pool row of
// every token, and tokens whose chunk an earlier sequence already filled are not written.
//
// One CTA per token: its angles go to shared memory once; then a group of lanes takes a head at a time, one 16-byte granule
// per lane (heads whose size or alignment does not allow that: a warp per head, one rotation pair per lane and step).  All arithmetic in fp32, one rounding at the store.  Heads are padded with zeros
// to whole 16-byte granules in the pool and in q, so that the attention kernels read granules for every head size.
#include <algorithm>

#include "ca_kernels.h"
#include "ca_types.cuh"

namespace ca {
namespace {

constexpr int QKV_WARPS = 4;
constexpr int QKV_MAX_D = 256;
constexpr int QKV_STEPS = QKV_MAX_D / 64;  // pairs a lane owns

template <typename T>
__global__ void __launch_bounds__(QKV_WARPS * 32) store_qkv_kernel(const QkvParams p) {
    __shared__ float2 turn_k[QKV_MAX_D / 2], turn_v[QKV_MAX_D / 2];  // (cos, sin) of every pair
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float pos = (float)p.positions[t];
    const int kp = p.key_freq ? p.rot_dims / 2 : 0, vp = p.value_freq ? p.d_value / 2 : 0;
    for (int i = threadIdx.x; i < kp + vp; i += blockDim.x) {
        float sn, cs;
        sincos_for<T>(pos * (i < kp ? p.key_freq[i] : p.value_freq[i - kp]), &sn, &cs);
        (i < kp ? turn_k[i] : turn_v[i - kp]) = make_float2(cs, sn);
    }
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
    __syncthreads();
    const int G = p.geo.n_heads, H = G * p.group;
    const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.row_stride;
    T* pool = reinterpret_cast<T*>(p.pool);
    const Geometry v_side = tile_side(p.geo, 1);
    for (int u = warp; u < H + 2 * G; u += QKV_WARPS) {
        const int kind = u < H ? 0 : (u < H + G ? 1 : 2);  // q, k, v
        const int h = kind == 0 ? u : (kind == 1 ? u - H : u - H - G);
        if (kind > 0 && chunk < 0) continue;
        const int d = kind == 2 ? p.d_value : p.d_key;
        const int padded = kind == 2 ? p.geo.d_value : p.geo.d_head;
        const T* src = row + (kind == 2 ? (H + G) * p.d_key + h * p.d_value : u * p.d_key);
        float a[QKV_STEPS], b[QKV_STEPS];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < QKV_STEPS; j++) {
            const int e = 2 * (lane + 32 * j);
            a[j] = e < d ? to_f32(src[e]) : 0.f;
            b[j] = e + 1 < d ? to_f32(src[e + 1]) : 0.f;
            ss = fmaf(a[j], a[j], fmaf(b[j], b[j], ss));
        }
        const float* w = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
        if (w) {
            const float inv = 1.f / sqrtf(warp_sum(ss) / d + p.eps);
#pragma unroll
            for (int j = 0; j < QKV_STEPS; j++) {
                const int e = 2 * (lane + 32 * j);
                if (e < d) a[j] = a[j] * inv * w[e];
                if (e + 1 < d) b[j] = b[j] * inv * w[e + 1];
            }
        }
        const int pairs = kind == 2 ? vp : kp;
        const float2* turn = kind == 2 ? turn_v : turn_k;
        T* dst;
        Geometry side = p.geo;
        if (kind == 0) {
            dst = reinterpret_cast<T*>(p.q_out) + ((size_t)t * H + h) * padded;
        } else {
            if (kind == 2) side = v_side;
            dst = pool + tile_base_elems(p.geo, chunk, h, kind - 1);
        }
#pragma unroll
        for (int j = 0; j < QKV_STEPS; j++) {
            const int i = lane + 32 * j, e = 2 * i;
            if (e >= padded) break;
            if (i < pairs) {
                const float2 cs = turn[i];
                const float x = a[j], y = b[j];
                a[j] = x * cs.x - y * cs.y;
                b[j] = y * cs.x + x * cs.y;
            }
            // a pair never straddles two granules, and padded rows have an even number of elements
            const int64_t off = kind == 0 ? e : tile_elem_offset(side, slot, e);
            Pack<T, 2> o;
            o.v[0] = from_f32<T>(a[j]);
            o.v[1] = from_f32<T>(b[j]);
            *reinterpret_cast<Pack<T, 2>*>(dst + off) = o;
        }
    }
}

// Heads of whole granules, up to `lanes` of them (a power of two, at most 32).
constexpr int QKV_VEC_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(QKV_VEC_THREADS) store_qkv_vec_kernel(const QkvParams p, int lanes) {
    constexpr int EPG = 16 / sizeof(T), PPG = EPG / 2;
    __shared__ float2 turn_k[QKV_MAX_D / 2], turn_v[QKV_MAX_D / 2];  // (cos, sin) of every pair
    const int t = blockIdx.x, tid = threadIdx.x;
    const float pos = (float)p.positions[t];
    const int kp = p.key_freq ? p.rot_dims / 2 : 0, vp = p.value_freq ? p.d_value / 2 : 0;
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
    const int G = p.geo.n_heads, H = G * p.group, units = H + 2 * G;
    const int g = tid & (lanes - 1), per_pass = QKV_VEC_THREADS / lanes;
    const T* row = reinterpret_cast<const T*>(p.qkv) + (size_t)t * p.row_stride;
    T* pool = reinterpret_cast<T*>(p.pool);
    const Geometry v_side = tile_side(p.geo, 1);
    constexpr int AHEAD = 1;  // heads whose granules are requested together
    Pack<T, EPG> in[AHEAD];
    auto source = [&](int u) { return row + (u < H + G ? u * p.d_key : (H + G) * p.d_key + (u - H - G) * p.d_value) + g * EPG; };
    auto size_of = [&](int u) { return u < H + G ? p.d_key : p.d_value; };
    int u = tid / lanes;
    auto request = [&](int u) {
#pragma unroll
        for (int a = 0; a < AHEAD; a++) {
            const int ua = u + a * per_pass;
            if (ua < units && g * EPG < size_of(ua)) in[a] = *reinterpret_cast<const Pack<T, EPG>*>(source(ua));
        }
    };
    request(u);
    for (int i = tid; i < kp + vp; i += QKV_VEC_THREADS) {
        float sn, cs;
        sincos_for<T>(pos * (i < kp ? p.key_freq[i] : p.value_freq[i - kp]), &sn, &cs);
        (i < kp ? turn_k[i] : turn_v[i - kp]) = make_float2(cs, sn);
    }
    __syncthreads();
    auto one_head = [&](int u, const Pack<T, EPG>& in) {
        const bool on = u < units && g * EPG < size_of(min(u, units - 1));
        const int kind = u < H ? 0 : (u < H + G ? 1 : 2);  // q, k, v
        float x[EPG];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < EPG; i++) {
            x[i] = on ? to_f32(in.v[i]) : 0.f;
            ss = fmaf(x[i], x[i], ss);
        }
        for (int off = lanes >> 1; off >= 1; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
        if (!on || (kind > 0 && chunk < 0)) return;
        const float* w = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
        if (w) {
            const float inv = 1.f / sqrtf(ss / p.d_key + p.eps);
#pragma unroll
            for (int i = 0; i < EPG; i += 4) {
                const float4 ww = *reinterpret_cast<const float4*>(w + g * EPG + i);
                x[i] *= inv * ww.x;
                x[i + 1] *= inv * ww.y;
                x[i + 2] *= inv * ww.z;
                x[i + 3] *= inv * ww.w;
            }
        }
        const float2* turn = (kind == 2 ? turn_v : turn_k) + g * PPG;
        const int pairs = (kind == 2 ? vp : kp) - g * PPG;
#pragma unroll
        for (int i = 0; i < PPG; i++)
            if (i < pairs) {
                const float2 cs = turn[i];
                const float a = x[2 * i], b = x[2 * i + 1];
                x[2 * i] = a * cs.x - b * cs.y;
                x[2 * i + 1] = b * cs.x + a * cs.y;
            }
        Pack<T, EPG> o;
#pragma unroll
        for (int i = 0; i < EPG; i++) o.v[i] = from_f32<T>(x[i]);
        Pack<T, EPG>* dst;
        if (kind == 0) {
            dst = reinterpret_cast<Pack<T, EPG>*>(reinterpret_cast<T*>(p.q_out) + ((size_t)t * H + u) * p.geo.d_head) + g;
        } else {
            const int h = u - (kind == 1 ? H : H + G);
            dst = reinterpret_cast<Pack<T, EPG>*>(pool + tile_base_elems(p.geo, chunk, h, kind - 1)) +
                  tile_granule_index(kind == 2 ? v_side : p.geo, slot, g);
        }
        *dst = o;
    };
    for (int u0 = 0; u0 < units; u0 += AHEAD * per_pass, u += AHEAD * per_pass) {
        if (u0 > 0) request(u);
#pragma unroll
        for (int a = 0; a < AHEAD; a++) one_head(u + a * per_pass, in[a]);
    }
}
template <typename T>
void run_store_qkv(const QkvParams& p, cudaStream_t stream) {
    constexpr int EPG = 16 / sizeof(T);
    auto aligned = [](const void* q) { return reinterpret_cast<uintptr_t>(q) % 16 == 0; };
    const int granules = std::max(p.d_key, p.d_value) / EPG;
    if (p.d_key % EPG == 0 && p.d_value % EPG == 0 && p.row_stride % EPG == 0 && aligned(p.qkv) && aligned(p.q_norm) && aligned(p.k_norm) &&
        granules <= 32) {
        int lanes = 1;
        while (lanes < granules) lanes *= 2;
        store_qkv_vec_kernel<T><<<p.n_tokens, QKV_VEC_THREADS, 0, stream>>>(p, lanes);
    } else {
        store_qkv_kernel<T><<<p.n_tokens, QKV_WARPS * 32, 0, stream>>>(p);
    }
}

}  // namespace

cudaError_t launch_store_qkv(const QkvParams& p, int dtype, cudaStream_t stream) {
    if (p.n_tokens <= 0) return cudaSuccess;
    if (p.geo.d_head > QKV_MAX_D || p.geo.d_value > QKV_MAX_D || p.geo.epg < 2) return cudaErrorInvalidValue;
    if (dtype == 2) run_store_qkv<__nv_bfloat16>(p, stream);
    else if (dtype == 1) run_store_qkv<float>(p, stream);
    else run_store_qkv<__half>(p, stream);
    return cudaGetLastError();
}

}  // namespace ca
