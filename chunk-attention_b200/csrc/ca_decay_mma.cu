// Linear attention with a per-head decay over spans, on tensor cores (bf16, mma.sync): S <- d S + k v^T, o = S^T q.
//
// A CTA takes one head and one run of 64-token blocks.  For a block of n tokens and the state S0 before it
//   P    = (Q K^T) * d^(i - j), j <= i          scores, fp32, masked and decayed
//   O    = P V + d^(i + 1) Q S0
//   S    = d^n S0 + (d^(n - 1 - j) K)^T V
// S lives in fp32 accumulators for the whole run; before each block its value goes to shared memory as bf16 hi + lo parts for
// the product with Q.  P and the decayed K enter their products as hi + lo parts too, so the decays, the scores and the
// state keep 16 bits or more while every multiplication runs on tensor cores.
// Eight warps: for P and O warp w has rows 16 (w & 3) .. and half of the value columns; for S a 16-row tile of the keys.
#include "ca_kernels.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
namespace {
using namespace ptx;

constexpr int D_THREADS = 256, D_TOK = 64;

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
__device__ __forceinline__ float lo_f(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float hi_f(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16(a, b);
    lo = pack_bf16(a - lo_f(hi), b - hi_f(hi));
}
// byte offset of granule g of row r in a matrix of ROWS rows stored as 128-byte panels, granules XOR-ed with the row
template <int ROWS> __device__ __forceinline__ uint32_t at(int r, int g) { return (g >> 3) * (ROWS * 128) + r * 128 + (((g & 7) ^ (r & 7)) << 4); }

template <int DK, int DV> struct Smem {
    static constexpr int Q = 0, K = Q + D_TOK * DK * 2, V = K + D_TOK * DK * 2, S_HI = V + D_TOK * DV * 2, S_LO = S_HI + DK * DV * 2,
                         PW = S_LO + DK * DV * 2, BYTES = PW + (D_TOK + 1) * 4;
};

// PHASE 0: the span is one run: state in, outputs, state out.  1: end state of the run from zero.  2: outputs from the run's
// initial state.
template <int DK, int DV, int PHASE>
__global__ void __launch_bounds__(D_THREADS, 1) decay_mma_kernel(const DecayMmaParams p) {
    using M = Smem<DK, DV>;
    constexpr int WR = DK / 16, CW = 8 / WR, NTS = DV / CW / 8;  // state: row tiles, column groups, n-tiles of a warp
    constexpr int NTO = DV / 16;                                // output n-tiles of a warp (half of the columns)
    extern __shared__ __align__(1024) uint8_t smem[];
    const uint32_t sb = smem_u32(smem);
    float* pw = reinterpret_cast<float*>(smem + M::PW);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, mat = lane >> 3, r8 = lane & 7, quad = lane >> 2, q2 = (lane & 3) * 2;
    const int h = blockIdx.x;
    int e, t_begin, t_end, piece = blockIdx.y;
    if (PHASE == 0) {
        e = blockIdx.y;
        t_begin = p.sp.cu[e];
        t_end = p.sp.cu[e + 1];
    } else {
        const int4 wk = reinterpret_cast<const int4*>(p.sp.work)[piece];
        if (wk.w % p.run) return;  // a run starts at every run-th piece
        e = wk.x;
        t_begin = wk.y;
        t_end = min(p.sp.cu[e + 1], t_begin + p.run * p.sp.work_len);
    }
    const float d = p.decay[h];
    for (int i = tid; i <= D_TOK; i += D_THREADS) pw[i] = powf(d, (float)i);

    const int sr = (warp % WR) * 16, sc = (warp / WR) * (DV / CW);  // this warp's tile of the state
    float S[NTS][4];
    float* slot = p.state + ((size_t)p.sp.slot[e] * p.H + h) * p.dk * p.dv;
    float* local = p.piece_state + ((size_t)piece * p.H + h) * p.dk * p.dv;
    const bool load = PHASE == 2 || (PHASE == 0 && p.sp.start[e] > 0);
    const float* src = PHASE == 2 ? local : slot;
#pragma unroll
    for (int nt = 0; nt < NTS; nt++)
#pragma unroll
        for (int k = 0; k < 4; k++) {
            const int row = sr + quad + 8 * (k >> 1), col = sc + 8 * nt + q2 + (k & 1);
            S[nt][k] = load && row < p.dk && col < p.dv ? src[(size_t)row * p.dv + col] : 0.f;
        }

    const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(p.qkv);
    const int Hk = p.H * p.dk;
    auto fill = [&](uint32_t dst, int width, int padded, int offset, int t0, int n) {
        const int gr = padded / 8;
        for (int i = tid; i < D_TOK * gr; i += D_THREADS) {
            const int t = i / gr, g = i % gr;
            uint32_t o[4] = {0u, 0u, 0u, 0u};
            if (t < n && g * 8 < width) {
                const uint4 v = __ldg(reinterpret_cast<const uint4*>(qkv + (size_t)(t0 + t) * p.row_stride + offset) + g);
                const uint32_t x[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
                for (int k = 0; k < 4; k++) o[k] = pack_bf16(silu_for<__nv_bfloat16>(lo_f(x[k])), silu_for<__nv_bfloat16>(hi_f(x[k])));
            }
            sts128(dst + at<D_TOK>(t, g), (int)o[0], (int)o[1], (int)o[2], (int)o[3]);
        }
    };

    const int rt = (warp & 3) * 16, oc = (warp >> 2) * (DV / 2);  // output rows and first column of this warp
    for (int t0 = t_begin; t0 < t_end; t0 += D_TOK) {
        const int n = min(D_TOK, t_end - t0);
        __syncthreads();
        if (PHASE != 1) fill(sb + M::Q, p.dk, DK, h * p.dk, t0, n);
        fill(sb + M::K, p.dk, DK, Hk + h * p.dk, t0, n);
        fill(sb + M::V, p.dv, DV, 2 * Hk + h * p.dv, t0, n);
        if (PHASE != 1) {
#pragma unroll
            for (int nt = 0; nt < NTS; nt++)
#pragma unroll
                for (int k = 0; k < 2; k++) {
                    uint32_t hi, lo;
                    split_bf16(S[nt][2 * k], S[nt][2 * k + 1], hi, lo);
                    const int row = sr + quad + 8 * k, col = sc + 8 * nt;
                    const uint32_t off = at<DK>(row, col >> 3) + q2 * 2;
                    *reinterpret_cast<uint32_t*>(smem + M::S_HI + off) = hi;
                    *reinterpret_cast<uint32_t*>(smem + M::S_LO + off) = lo;
                }
        }
        __syncthreads();

        if (PHASE != 1) {
            float o[NTO][4];
#pragma unroll
            for (int i = 0; i < NTO; i++)
#pragma unroll
                for (int k = 0; k < 4; k++) o[i][k] = 0.f;
            // Q S0
#pragma unroll
            for (int ks = 0; ks < DK / 16; ks++) {
                uint32_t a[4];
                ldsm_x4(a[0], a[1], a[2], a[3], sb + M::Q + at<D_TOK>(rt + (mat & 1) * 8 + r8, 2 * ks + (mat >> 1)));
#pragma unroll
                for (int part = 0; part < 2; part++)
#pragma unroll
                    for (int dt = 0; dt < NTO / 2; dt++) {
                        uint32_t b0, b1, b2, b3;
                        ldsm_x4_trans(b0, b1, b2, b3, sb + (part ? M::S_LO : M::S_HI) + at<DK>(16 * ks + (mat & 1) * 8 + r8, (oc >> 3) + 2 * dt + (mat >> 1)));
                        mma_bf16(o[2 * dt], a, b0, b1);
                        mma_bf16(o[2 * dt + 1], a, b2, b3);
                    }
            }
            const float f0 = pw[rt + quad + 1], f1 = pw[rt + quad + 9 > D_TOK ? D_TOK : rt + quad + 9];
#pragma unroll
            for (int i = 0; i < NTO; i++) {
                o[i][0] *= f0;
                o[i][1] *= f0;
                o[i][2] *= f1;
                o[i][3] *= f1;
            }
            // P V, 16 tokens at a time, up to the diagonal
            for (int sl = 0; sl <= (rt >> 4); sl++) {
                float s[2][4];
#pragma unroll
                for (int i = 0; i < 2; i++)
#pragma unroll
                    for (int k = 0; k < 4; k++) s[i][k] = 0.f;
#pragma unroll
                for (int ks = 0; ks < DK / 16; ks++) {
                    uint32_t a[4], b0, b1, b2, b3;
                    ldsm_x4(a[0], a[1], a[2], a[3], sb + M::Q + at<D_TOK>(rt + (mat & 1) * 8 + r8, 2 * ks + (mat >> 1)));
                    ldsm_x4(b0, b1, b2, b3, sb + M::K + at<D_TOK>(16 * sl + (mat >> 1) * 8 + r8, 2 * ks + (mat & 1)));
                    mma_bf16(s[0], a, b0, b1);
                    mma_bf16(s[1], a, b2, b3);
                }
#pragma unroll
                for (int i = 0; i < 2; i++)
#pragma unroll
                    for (int k = 0; k < 4; k++) {
                        const int dist = rt + quad + 8 * (k >> 1) - (16 * sl + 8 * i + q2 + (k & 1));
                        s[i][k] = dist >= 0 ? s[i][k] * pw[dist] : 0.f;
                    }
                uint32_t hi[4], lo[4];
                split_bf16(s[0][0], s[0][1], hi[0], lo[0]);
                split_bf16(s[0][2], s[0][3], hi[1], lo[1]);
                split_bf16(s[1][0], s[1][1], hi[2], lo[2]);
                split_bf16(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
                for (int dt = 0; dt < NTO / 2; dt++) {
                    uint32_t b0, b1, b2, b3;
                    ldsm_x4_trans(b0, b1, b2, b3, sb + M::V + at<D_TOK>(16 * sl + (mat & 1) * 8 + r8, (oc >> 3) + 2 * dt + (mat >> 1)));
                    mma_bf16(o[2 * dt], hi, b0, b1);
                    mma_bf16(o[2 * dt], lo, b0, b1);
                    mma_bf16(o[2 * dt + 1], hi, b2, b3);
                    mma_bf16(o[2 * dt + 1], lo, b2, b3);
                }
            }
            __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
#pragma unroll
            for (int k = 0; k < 2; k++) {
                const int row = rt + quad + 8 * k;
                if (row < n) {
                    __nv_bfloat16* dst = out + ((size_t)(t0 + row) * p.H + h) * p.dv;
#pragma unroll
                    for (int i = 0; i < NTO; i++) {
                        const int col = oc + 8 * i + q2;
                        if (col < p.dv) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16(o[i][2 * k], o[i][2 * k + 1]);
                    }
                }
            }
        }
        if (PHASE == 2 && t0 + D_TOK >= t_end) break;
        // S = d^n S + (d^(n-1-j) K)^T V
        const float dn = pw[n];
#pragma unroll
        for (int nt = 0; nt < NTS; nt++)
#pragma unroll
            for (int k = 0; k < 4; k++) S[nt][k] *= dn;
#pragma unroll
        for (int ks = 0; ks < D_TOK / 16; ks++) {
            if (16 * ks >= n) break;
            // A = K^T: rows are key elements, the contraction runs over tokens
            uint32_t a[4], hi[4], lo[4];
            ldsm_x4_trans(a[0], a[1], a[2], a[3], sb + M::K + at<D_TOK>(16 * ks + (mat >> 1) * 8 + r8, (sr >> 3) + (mat & 1)));
#pragma unroll
            for (int k = 0; k < 4; k++) {
                const int j = 16 * ks + (k >> 1) * 8 + q2;
                split_bf16(lo_f(a[k]) * pw[max(n - 1 - j, 0)], hi_f(a[k]) * pw[max(n - 2 - j, 0)], hi[k], lo[k]);
            }
#pragma unroll
            for (int dt = 0; dt < NTS / 2; dt++) {
                uint32_t b0, b1, b2, b3;
                ldsm_x4_trans(b0, b1, b2, b3, sb + M::V + at<D_TOK>(16 * ks + (mat & 1) * 8 + r8, (sc >> 3) + 2 * dt + (mat >> 1)));
                mma_bf16(S[2 * dt], hi, b0, b1);
                mma_bf16(S[2 * dt], lo, b0, b1);
                mma_bf16(S[2 * dt + 1], hi, b2, b3);
                mma_bf16(S[2 * dt + 1], lo, b2, b3);
            }
        }
    }
    if (PHASE == 2) return;
    float* dst = PHASE == 0 ? slot : local;
#pragma unroll
    for (int nt = 0; nt < NTS; nt++)
#pragma unroll
        for (int k = 0; k < 2; k++) {
            const int row = sr + quad + 8 * k, col = sc + 8 * nt + q2;
            if (row < p.dk && col < p.dv) *reinterpret_cast<float2*>(dst + (size_t)row * p.dv + col) = make_float2(S[nt][2 * k], S[nt][2 * k + 1]);
        }
}

// end states of the runs -> initial states, and the span's end state to its slot
__global__ void decay_sweep_kernel(const DecayMmaParams p) {
    const int e = blockIdx.y;
    const int64_t per_head = (int64_t)p.dk * p.dv, all = per_head * p.H;
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
    if (i >= all) return;
    const float d = p.decay[i / per_head];
    float4* slot = reinterpret_cast<float4*>(p.state + (size_t)p.sp.slot[e] * all + i);
    float4 S = p.sp.start[e] > 0 ? *slot : make_float4(0.f, 0.f, 0.f, 0.f);
    const int end = p.sp.cu[e + 1], full = p.run * p.sp.work_len;
    const float d_full = powf(d, (float)full);
    constexpr int AHEAD = 8;  // runs requested together
    const int w_end = p.sp.work_off[e + 1];
    int t = p.sp.cu[e];
    for (int w0 = p.sp.work_off[e]; w0 < w_end; w0 += AHEAD * p.run) {
        float4 local[AHEAD];
#pragma unroll
        for (int k = 0; k < AHEAD; k++)
            if (w0 + k * p.run < w_end) local[k] = *reinterpret_cast<const float4*>(p.piece_state + (size_t)(w0 + k * p.run) * all + i);
#pragma unroll
        for (int k = 0; k < AHEAD; k++) {
            if (w0 + k * p.run >= w_end) break;
            const float f = end - t >= full ? d_full : powf(d, (float)(end - t));
            *reinterpret_cast<float4*>(p.piece_state + (size_t)(w0 + k * p.run) * all + i) = S;
            S = make_float4(fmaf(f, S.x, local[k].x), fmaf(f, S.y, local[k].y), fmaf(f, S.z, local[k].z), fmaf(f, S.w, local[k].w));
            t += full;
        }
    }
    *slot = S;
}

template <int DK, int DV, int PHASE>
cudaError_t launch_phase(const DecayMmaParams& p, int grid_y, cudaStream_t stream) {
    constexpr int smem = Smem<DK, DV>::BYTES;
    auto* k = decay_mma_kernel<DK, DV, PHASE>;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    k<<<dim3(p.H, grid_y), D_THREADS, smem, stream>>>(p);
    return cudaGetLastError();
}

template <int DK, int DV>
cudaError_t launch(const DecayMmaParams& p, cudaStream_t stream) {
    if (p.run == 0) return launch_phase<DK, DV, 0>(p, p.sp.n_entries, stream);
    cudaError_t e = launch_phase<DK, DV, 1>(p, p.sp.n_work, stream);
    if (e != cudaSuccess) return e;
    e = launch_decay_sweep(p, stream);
    if (e != cudaSuccess) return e;
    return launch_phase<DK, DV, 2>(p, p.sp.n_work, stream);
}

}  // namespace

cudaError_t launch_decay_sweep(const DecayMmaParams& p, cudaStream_t stream) {
    const int64_t quads = (int64_t)p.H * p.dk * p.dv / 4;
    decay_sweep_kernel<<<dim3((unsigned)((quads + 255) / 256), p.sp.n_entries), 256, 0, stream>>>(p);
    return cudaGetLastError();
}

bool decay_mma_serves(int dk, int dv, int64_t row_stride, const void* qkv, int work_len) {
    return dk % 16 == 0 && dv % 16 == 0 && dk <= 128 && dv <= 128 && row_stride % 8 == 0 && reinterpret_cast<uintptr_t>(qkv) % 16 == 0 &&
           work_len % D_TOK == 0;
}

cudaError_t launch_decay_mma(const DecayMmaParams& p, cudaStream_t stream) {
    if (p.dk <= 64) return p.dv <= 64 ? launch<64, 64>(p, stream) : launch<64, 128>(p, stream);
    return p.dv <= 64 ? launch<128, 64>(p, stream) : launch<128, 128>(p, stream);
}

}  // namespace ca
