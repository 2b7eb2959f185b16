// Linear attention with a per-head decay over spans on the Blackwell tensor path: tcgen05.mma (bf16), accumulators and the
// recurrent state in tensor memory.  The same recurrence as ca_decay_mma.cu, in blocks of 128 tokens, for key sizes up to
// 128 and value sizes of 64 or 128 elements.
//
// A CTA takes one head and one run of blocks.  With S0 the state before a block of n tokens:
//   P  = Q K^T                     128 x 128, fp32 in TMEM; masked and decayed by the threads, written back as bf16 hi + lo
//   O1 = Q S0                      S0 as bf16 hi + lo parts in shared memory
//   O2 = P V                       A = P from TMEM
//   S  = d^n S0 + K'^T V           K' = d^(n-1-j) k_j as bf16 hi + lo parts; S stays in TMEM in fp32
//   out = O2 + d^(i+1) O1
// TMEM columns: P 0-127, O1 128-255, O2 256-383, S 384-511.  Shared memory: Q (later K' hi), K (later K' lo), V, S hi, S lo, each
// in the 128-byte-swizzled panels the matrix descriptors name.  Eight warps do the element work (warp w: lanes 32 (w & 3) ..,
// one half of the columns); one thread issues the MMAs; the next block's inputs are on their way in registers meanwhile.
// Both waits of a block are bounded: on expiry a status code is recorded and the CTA leaves through the common exit, which frees
// the TMEM columns.
#include "ca_kernels.h"
#include "ca_ptx.cuh"
#include "ca_types.cuh"

namespace ca {
__device__ int g_decay_status = 0;

namespace {
using namespace ptx;

constexpr int T_THREADS = 256, T_TOK = 128, T_DK = 128;
constexpr int T_PANEL = T_TOK * 128;                  // 64 elements of 128 rows
constexpr int T_MAT = 2 * T_PANEL;                    // a 128 x 128 bf16 matrix
constexpr uint32_t COL_P = 0, COL_O1 = 128, COL_O2 = 256, COL_S = 384;

template <int DV> struct Smem {
    static constexpr int Q = 0, K = Q + T_MAT, V = K + T_MAT, S_HI = V + (DV / 64) * T_PANEL, S_LO = S_HI + (DV / 64) * T_PANEL,
                         PW = S_LO + (DV / 64) * T_PANEL, BAR = PW + (T_TOK + 4) * 4, BYTES = BAR + 32;
};

__host__ __device__ constexpr uint32_t idesc_bf16(int m, int n, bool a_mn, bool b_mn) { return umma_idesc_f16(m, n, a_mn, b_mn) | (1u << 7) | (1u << 10); }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&h);
}
__device__ __forceinline__ float lo_f(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float hi_f(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
__device__ __forceinline__ uint32_t rest_bf16(float a, float b, uint32_t hi) { return pack_bf16(a - lo_f(hi), b - hi_f(hi)); }
// byte offset of granule g of row r in a matrix of 128 rows
__device__ __forceinline__ uint32_t at(int r, int g) { return (g >> 3) * T_PANEL + r * 128 + (((g & 7) ^ (r & 7)) << 4); }
__device__ __forceinline__ uint4 silu_granule(uint4 v) {
    uint32_t x[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int k = 0; k < 4; k++) x[k] = pack_bf16(silu_for<__nv_bfloat16>(lo_f(x[k])), silu_for<__nv_bfloat16>(hi_f(x[k])));
    return make_uint4(x[0], x[1], x[2], x[3]);
}
__device__ __forceinline__ void sts(uint32_t addr, uint4 v) { sts128(addr, (int)v.x, (int)v.y, (int)v.z, (int)v.w); }

// PHASE 0: the span is one run: state in, outputs, state out.  1: end state of the run from zero.  2: outputs from the run's
// initial state.
template <int DV, int PHASE>
__global__ void __launch_bounds__(T_THREADS, 1) decay_tc_kernel(const DecayMmaParams p) {
    using M = Smem<DV>;
    constexpr int KG = T_DK / 8, VG = DV / 8;                                   // granules of a row
    constexpr int KU = T_TOK * KG / T_THREADS, VU = T_TOK * VG / T_THREADS;     // granules of a thread
    constexpr int HALF = DV / 2;                                                // columns a thread handles of S and of the outputs
    extern __shared__ __align__(1024) uint8_t smem[];
    const uint32_t sb = smem_u32(smem);
    float* pw = reinterpret_cast<float*>(smem + M::PW);
    const uint32_t bar_qk = sb + M::BAR, bar_pv = bar_qk + 8;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(smem + M::BAR + 16);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row = 32 * (warp & 3) + lane, half = warp >> 2;
    const int h = blockIdx.x, piece = blockIdx.y;
    int e, t_begin, t_end;
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
    for (int i = tid; i <= T_TOK; i += T_THREADS) pw[i] = powf(d, (float)i);
    if (tid == 0) {
        mbar_init(bar_qk, 1);
        mbar_init(bar_pv, 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 0) {
        tmem_alloc(smem_u32(tmem_slot), 512);
        tmem_relinquish_alloc_permit();
    }
    tc_fence_before_thread_sync();
    __syncthreads();
    tc_fence_after_thread_sync();
    const uint32_t tmem = *tmem_slot;
    const uint32_t lanes = tmem + ((uint32_t)(32 * (warp & 3)) << 16);

    // ---- inputs: raw granules in registers, SiLU on the way to shared memory
    const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(p.qkv);
    const int Hk = p.H * p.dk;
    uint4 rq[PHASE == 1 ? 1 : KU], rk[KU], rv[VU];
    auto request = [&](int t0) {
        auto fetch = [&](int t, int g, int width, int offset) {
            if (t0 + t < t_end && g * 8 < width)
                return __ldg(reinterpret_cast<const uint4*>(qkv + (size_t)(t0 + t) * p.row_stride + offset) + g);
            return make_uint4(0u, 0u, 0u, 0u);
        };
#pragma unroll
        for (int u = 0; u < KU; u++) {
            const int i = tid + u * T_THREADS, t = i / KG, g = i % KG;
            if (PHASE != 1) rq[PHASE == 1 ? 0 : u] = fetch(t, g, p.dk, h * p.dk);
            rk[u] = fetch(t, g, p.dk, Hk + h * p.dk);
        }
#pragma unroll
        for (int u = 0; u < VU; u++) {
            const int i = tid + u * T_THREADS, t = i / VG, g = i % VG;
            rv[u] = fetch(t, g, p.dv, 2 * Hk + h * p.dv);
        }
    };
    request(t_begin);

    // ---- state: TMEM holds d^n S0 for the block that comes, shared memory the hi + lo parts of S0
    auto put_parts = [&](int c, const float* s) {  // 32 columns from c
#pragma unroll
        for (int g = 0; g < 4; g++) {
            uint32_t hi[4], lo[4];
#pragma unroll
            for (int k = 0; k < 4; k++) {
                hi[k] = pack_bf16(s[8 * g + 2 * k], s[8 * g + 2 * k + 1]);
                lo[k] = rest_bf16(s[8 * g + 2 * k], s[8 * g + 2 * k + 1], hi[k]);
            }
            const uint32_t off = at(row, (c >> 3) + g);
            sts128(sb + M::S_HI + off, (int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]);
            sts128(sb + M::S_LO + off, (int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]);
        }
    };
    float* slot = p.state + ((size_t)p.sp.slot[e] * p.H + h) * p.dk * p.dv;
    float* local = p.piece_state + ((size_t)piece * p.H + h) * p.dk * p.dv;
    {
        const bool load = PHASE == 2 || (PHASE == 0 && p.sp.start[e] > 0);
        const float* src = PHASE == 2 ? local : slot;
        const float dn = pw[min(T_TOK, t_end - t_begin)];
#pragma unroll
        for (int c = half * HALF; c < half * HALF + HALF; c += 32) {
            float s[32];
            uint32_t u[32];
#pragma unroll
            for (int k = 0; k < 32; k += 4) {
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                if (load && row < p.dk && c + k < p.dv) v = *reinterpret_cast<const float4*>(src + (size_t)row * p.dv + c + k);
                s[k] = v.x; s[k + 1] = v.y; s[k + 2] = v.z; s[k + 3] = v.w;
            }
#pragma unroll
            for (int k = 0; k < 32; k++) u[k] = __float_as_uint(s[k] * dn);
            if (PHASE != 1) put_parts(c, s);
            tmem_st32(lanes + COL_S + c, u);
        }
        tmem_wait_st();
    }

    constexpr uint32_t DESC_HI = umma_desc_sw128_hi(1024);
    constexpr uint32_t ID_QK = idesc_bf16(T_TOK, T_TOK, false, false), ID_OV = idesc_bf16(T_TOK, DV, false, true), ID_KV = idesc_bf16(T_DK, DV, true, true);
    bool ok = true;
    int b = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += T_TOK, b++) {
        const int n = min(T_TOK, t_end - t0);
        const bool more = t0 + T_TOK < t_end, update = PHASE != 2 || more;
        // ---- A: this block's operands
#pragma unroll
        for (int u = 0; u < KU; u++) {
            const int i = tid + u * T_THREADS, t = i / KG, g = i % KG;
            if (PHASE != 1) sts(sb + M::Q + at(t, g), silu_granule(rq[PHASE == 1 ? 0 : u]));
            if (PHASE != 1) {
                sts(sb + M::K + at(t, g), silu_granule(rk[u]));
            } else {
                // no scores here: K' right away
                const uint4 kv = silu_granule(rk[u]);
                const uint32_t x[4] = {kv.x, kv.y, kv.z, kv.w};
                uint32_t hi[4], lo[4];
                const float w = pw[max(n - 1 - t, 0)];
#pragma unroll
                for (int k = 0; k < 4; k++) {
                    hi[k] = pack_bf16(lo_f(x[k]) * w, hi_f(x[k]) * w);
                    lo[k] = rest_bf16(lo_f(x[k]) * w, hi_f(x[k]) * w, hi[k]);
                }
                sts128(sb + M::Q + at(t, g), (int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]);
                sts128(sb + M::K + at(t, g), (int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]);
            }
        }
#pragma unroll
        for (int u = 0; u < VU; u++) {
            const int i = tid + u * T_THREADS, t = i / VG, g = i % VG;
            sts(sb + M::V + at(t, g), silu_granule(rv[u]));
        }
        fence_proxy_async();
        tc_fence_before_thread_sync();
        __syncthreads();
        tc_fence_after_thread_sync();
        if (more) request(t0 + T_TOK);
        if (PHASE != 1) {
            // ---- B: P = Q K^T, O1 = Q S0
            if (warp == 0 && elect_one()) {
                const uint32_t q_lo = umma_desc_sw128_lo(sb + M::Q, 16), k_lo = umma_desc_sw128_lo(sb + M::K, 16);
#pragma unroll
                for (int ks = 0; ks < T_DK / 16; ks++) {
                    const uint32_t step = ((ks >> 2) * T_PANEL + (ks & 3) * 32) >> 4;
                    umma_ss_f16(tmem + COL_P, umma_desc_pack(q_lo + step, DESC_HI), umma_desc_pack(k_lo + step, DESC_HI), ID_QK, ks > 0 ? 1u : 0u);
                }
#pragma unroll
                for (int part = 0; part < 2; part++) {
                    const uint32_t s_lo = umma_desc_sw128_lo(sb + (part ? M::S_LO : M::S_HI), T_PANEL);
#pragma unroll
                    for (int ks = 0; ks < T_DK / 16; ks++) {
                        const uint32_t step = ((ks >> 2) * T_PANEL + (ks & 3) * 32) >> 4;
                        umma_ss_f16(tmem + COL_O1, umma_desc_pack(q_lo + step, DESC_HI), umma_desc_pack(s_lo + ((ks * 2048) >> 4), DESC_HI), ID_OV,
                                    (part > 0 || ks > 0) ? 1u : 0u);
                    }
                }
                umma_commit(bar_qk);
            }
            __syncwarp();
            ok = mbar_wait_bounded(bar_qk, b & 1, DEFAULT_WAIT_LIMIT_CYCLES);
            ok = __syncthreads_and(ok);
            if (!ok) break;
            tc_fence_after_thread_sync();
            // ---- C: decayed scores and decayed keys
            uint32_t s0[32], s1[32];
            tmem_ld32(lanes + COL_P + half * 64, s0);
            tmem_ld32(lanes + COL_P + half * 64 + 32, s1);
            if (update) {
#pragma unroll
                for (int u = 0; u < KU; u++) {
                    const int i = tid + u * T_THREADS, t = i / KG, g = i % KG;
                    const uint4 kv = lds128(sb + M::K + at(t, g));
                    const uint32_t x[4] = {kv.x, kv.y, kv.z, kv.w};
                    uint32_t hi[4], lo[4];
                    const float w = pw[max(n - 1 - t, 0)];
#pragma unroll
                    for (int k = 0; k < 4; k++) {
                        hi[k] = pack_bf16(lo_f(x[k]) * w, hi_f(x[k]) * w);
                        lo[k] = rest_bf16(lo_f(x[k]) * w, hi_f(x[k]) * w, hi[k]);
                    }
                    sts128(sb + M::Q + at(t, g), (int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]);
                    sts128(sb + M::K + at(t, g), (int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]);
                }
            }
            tmem_wait_ld();
            tc_fence_before_thread_sync();
            __syncthreads();  // every score has been read: its columns may be overwritten
            tc_fence_after_thread_sync();
            uint32_t pk[32];
#pragma unroll
            for (int k = 0; k < 32; k++) {
                const int i0 = row - (half * 64 + k), i1 = i0 - 32;
                s0[k] = __float_as_uint(i0 >= 0 ? __uint_as_float(s0[k]) * pw[i0] : 0.f);
                s1[k] = __float_as_uint(i1 >= 0 ? __uint_as_float(s1[k]) * pw[i1] : 0.f);
            }
#pragma unroll
            for (int k = 0; k < 16; k++) {
                pk[k] = pack_bf16(__uint_as_float(s0[2 * k]), __uint_as_float(s0[2 * k + 1]));
                pk[16 + k] = pack_bf16(__uint_as_float(s1[2 * k]), __uint_as_float(s1[2 * k + 1]));
            }
            tmem_st32(lanes + COL_P + half * 32, pk);
#pragma unroll
            for (int k = 0; k < 16; k++) {
                pk[k] = rest_bf16(__uint_as_float(s0[2 * k]), __uint_as_float(s0[2 * k + 1]), pk[k]);
                pk[16 + k] = rest_bf16(__uint_as_float(s1[2 * k]), __uint_as_float(s1[2 * k + 1]), pk[16 + k]);
            }
            tmem_st32(lanes + COL_P + 64 + half * 32, pk);
            tmem_wait_st();
            fence_proxy_async();
            tc_fence_before_thread_sync();
            __syncthreads();
            tc_fence_after_thread_sync();
        }
        // ---- D: O2 = P V, S += K'^T V
        if (warp == 0 && elect_one()) {
            const uint32_t v_lo = umma_desc_sw128_lo(sb + M::V, T_PANEL);
            if (PHASE != 1) {
#pragma unroll
                for (int part = 0; part < 2; part++)
#pragma unroll
                    for (int ks = 0; ks < T_TOK / 16; ks++)
                        umma_ts_f16(tmem + COL_O2, tmem + COL_P + part * 64 + ks * 8, umma_desc_pack(v_lo + ((ks * 2048) >> 4), DESC_HI), ID_OV,
                                    (part > 0 || ks > 0) ? 1u : 0u);
            }
            if (update) {
#pragma unroll
                for (int part = 0; part < 2; part++) {
                    const uint32_t k_lo = umma_desc_sw128_lo(sb + (part ? M::K : M::Q), T_PANEL);
#pragma unroll
                    for (int ks = 0; ks < T_TOK / 16; ks++)
                        umma_ss_f16(tmem + COL_S, umma_desc_pack(k_lo + ((ks * 2048) >> 4), DESC_HI), umma_desc_pack(v_lo + ((ks * 2048) >> 4), DESC_HI), ID_KV, 1u);
                }
            }
            umma_commit(bar_pv);
        }
        __syncwarp();
        ok = mbar_wait_bounded(bar_pv, b & 1, DEFAULT_WAIT_LIMIT_CYCLES);
        ok = __syncthreads_and(ok);
        if (!ok) break;
        tc_fence_after_thread_sync();
        // ---- E: rows out, state for the next block
        if (PHASE != 1) {
            const float f = pw[min(row + 1, T_TOK)];
            __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + ((size_t)(t0 + row) * p.H + h) * p.dv;
#pragma unroll
            for (int c = half * HALF; c < half * HALF + HALF; c += 32) {
                uint32_t o1[32], o2[32];
                tmem_ld32(lanes + COL_O1 + c, o1);
                tmem_ld32(lanes + COL_O2 + c, o2);
                tmem_wait_ld();
                if (row < n) {
#pragma unroll
                    for (int g = 0; g < 4; g++) {
                        uint32_t o[4];
#pragma unroll
                        for (int k = 0; k < 4; k++) {
                            const int x = 8 * g + 2 * k;
                            o[k] = pack_bf16(fmaf(f, __uint_as_float(o1[x]), __uint_as_float(o2[x])), fmaf(f, __uint_as_float(o1[x + 1]), __uint_as_float(o2[x + 1])));
                        }
                        if (c + 8 * g < p.dv) *reinterpret_cast<uint4*>(dst + c + 8 * g) = make_uint4(o[0], o[1], o[2], o[3]);
                    }
                }
            }
        }
        if (update) {
            const float dn = more ? pw[min(T_TOK, t_end - t0 - T_TOK)] : 1.f;
            float* out = PHASE == 0 ? slot : local;
#pragma unroll
            for (int c = half * HALF; c < half * HALF + HALF; c += 32) {
                uint32_t u[32];
                float s[32];
                tmem_ld32(lanes + COL_S + c, u);
                tmem_wait_ld();
#pragma unroll
                for (int k = 0; k < 32; k++) s[k] = __uint_as_float(u[k]);
                if (more) {
                    if (PHASE != 1) put_parts(c, s);
#pragma unroll
                    for (int k = 0; k < 32; k++) u[k] = __float_as_uint(s[k] * dn);
                    tmem_st32(lanes + COL_S + c, u);
                } else if (row < p.dk) {
#pragma unroll
                    for (int k = 0; k < 32; k += 4)
                        if (c + k < p.dv) *reinterpret_cast<float4*>(out + (size_t)row * p.dv + c + k) = make_float4(s[k], s[k + 1], s[k + 2], s[k + 3]);
                }
            }
            tmem_wait_st();
        }
    }
    if (!ok && tid == 0) atomicCAS(&g_decay_status, STATUS_OK, STATUS_FULL_WAIT_TIMEOUT);
    // ---- common exit: nobody touches TMEM after this barrier, then the allocating warp frees it
    tc_fence_before_thread_sync();
    __syncthreads();
    if (warp == 0) {
        tc_fence_after_thread_sync();
        tmem_dealloc(tmem, 512);
    }
}

template <int DV, int PHASE>
cudaError_t launch_phase(const DecayMmaParams& p, int grid_y, cudaStream_t stream) {
    constexpr int smem = Smem<DV>::BYTES;
    auto* k = decay_tc_kernel<DV, PHASE>;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    k<<<dim3(p.H, grid_y), T_THREADS, smem, stream>>>(p);
    return cudaGetLastError();
}

template <int DV>
cudaError_t launch(const DecayMmaParams& p, cudaStream_t stream) {
    if (p.run == 0) return launch_phase<DV, 0>(p, p.sp.n_entries, stream);
    cudaError_t e = launch_phase<DV, 1>(p, p.sp.n_work, stream);
    if (e == cudaSuccess) e = launch_decay_sweep(p, stream);
    if (e == cudaSuccess) e = launch_phase<DV, 2>(p, p.sp.n_work, stream);
    return e;
}

}  // namespace

bool decay_tc_serves(int dk, int dv) { return dk <= T_DK && dv <= 128 && dk >= 48 && dv >= 32; }

cudaError_t launch_decay_tc(const DecayMmaParams& p, cudaStream_t stream) { return p.dv <= 64 ? launch<64>(p, stream) : launch<128>(p, stream); }

cudaError_t read_decay_status(int* status, cudaStream_t stream) {
    cudaError_t e = cudaMemcpyFromSymbolAsync(status, g_decay_status, sizeof(int), 0, cudaMemcpyDeviceToHost, stream);
    return e == cudaSuccess ? cudaStreamSynchronize(stream) : e;
}

}  // namespace ca
