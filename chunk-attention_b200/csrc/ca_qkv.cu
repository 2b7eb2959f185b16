// From the projections of a batch of tokens to attention operands, in one kernel: per-head RMS norm of q and k,
// rotation of q and k (interleaved pairs, a leading part of each head), rotation of v by its position, and the
// store - q to a dense buffer, k and v straight into the token's row of the chunk pool.  A decode step writes row
// s of the batch into the next free row of sequence s's tail chunk; a portion of a prompt names the pool row of
// every token, and tokens whose chunk an earlier sequence already filled are not written.
//
// One CTA per token: its angles go to shared memory once, then a warp takes a head at a time, 2 elements (one
// rotation pair) per lane and step.  All arithmetic in fp32, one rounding at the store.  Heads are padded with zeros
// to whole 16-byte granules in the pool and in q, so that the attention kernels read granules for every head size.
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
        sincosf(pos * (i < kp ? p.key_freq[i] : p.value_freq[i - kp]), &sn, &cs);
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

}  // namespace

cudaError_t launch_store_qkv(const QkvParams& p, int dtype, cudaStream_t stream) {
    if (p.n_tokens <= 0) return cudaSuccess;
    if (p.geo.d_head > QKV_MAX_D || p.geo.d_value > QKV_MAX_D || p.geo.epg < 2) return cudaErrorInvalidValue;
    if (dtype == 2) store_qkv_kernel<__nv_bfloat16><<<p.n_tokens, QKV_WARPS * 32, 0, stream>>>(p);
    else if (dtype == 1) store_qkv_kernel<float><<<p.n_tokens, QKV_WARPS * 32, 0, stream>>>(p);
    else store_qkv_kernel<__half><<<p.n_tokens, QKV_WARPS * 32, 0, stream>>>(p);
    return cudaGetLastError();
}

}  // namespace ca
