// Recurrent sequence mixers over batches of spans (consecutive tokens of several sequences, each with a state slot):
// causal depthwise convolution + SiLU, the selective scan of Mamba, and linear attention with a per-head decay.
// States are fp32, live in [slots][...] arrays of the caller, and are read at a span's start (taken as zero at position
// 0, so a slot needs no clearing before it is used again) and written at its end.
//
// The work of a step is listed as PIECES of at most `work_len` tokens of one span (ca_spans).  A step whose spans are
// all single pieces runs a recurrence in one launch; otherwise the scan takes three: local end state of every piece
// from zero, a sweep over the pieces of each sequence that turns them into initial states, and the outputs.
#include <algorithm>
#include <type_traits>

#include "../../include/chunk_attn_b200.h"
#include "ca_kernels.h"
#include "ca_types.cuh"

namespace ca {
namespace {

int fail(const char* msg, int code = CA_ERR_INVALID) {
    set_last_error(msg);
    return code;
}
int done() {
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? CA_OK : fail(cudaGetErrorString(e), CA_ERR_CUDA);
}
constexpr float LOG2E = 1.4426950408889634f;

// ---- convolution ------------------------------------------------------------------------------------------------
// A thread owns V channels and one piece.  KMAX - 1 previous inputs sit in registers, oldest first; a filter with
// fewer taps is right-aligned.  The thread of a span's first piece reads the state and, having read it, puts the
// span's last inputs back.
template <typename T, int V, int KMAX>
__global__ void __launch_bounds__(128) conv_silu_kernel(T* __restrict__ out, const T* __restrict__ x, int64_t x_stride,
                                                        const float* __restrict__ taps, const float* __restrict__ bias,
                                                        float* __restrict__ state, const ca_spans sp, int channels, int K) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (c >= channels) return;
    const int4 wk = reinterpret_cast<const int4*>(sp.work)[blockIdx.y];
    const int e = wk.x, t0 = wk.y, t1 = wk.z, first = sp.cu[e], last = sp.cu[e + 1];
    float tap[KMAX][V], hist[KMAX][V], b[V];
#pragma unroll
    for (int j = 0; j < KMAX; j++)
#pragma unroll
        for (int v = 0; v < V; v++) tap[j][v] = j >= KMAX - K ? taps[(size_t)(c + v) * K + j - (KMAX - K)] : 0.f;
#pragma unroll
    for (int v = 0; v < V; v++) b[v] = bias[c + v];
    float* st = state + (size_t)sp.slot[e] * (K - 1) * channels + c;
    const bool live = sp.start[e] > 0;
    // input at offset i from the span's first token, reaching back into the state
    auto input = [&](int i, float (&o)[V]) {
        if (i >= 0) {
            const Pack<T, V> a = *reinterpret_cast<const Pack<T, V>*>(x + (size_t)(first + i) * x_stride + c);
#pragma unroll
            for (int v = 0; v < V; v++) o[v] = to_f32(a.v[v]);
        } else {
#pragma unroll
            for (int v = 0; v < V; v++) o[v] = live ? st[(size_t)(i + K - 1) * channels + v] : 0.f;
        }
    };
    const int off = t0 - first;
#pragma unroll
    for (int j = 0; j < KMAX - 1; j++) {
        if (j >= KMAX - K) {
            input(off - (KMAX - 1) + j, hist[j]);
        } else {
#pragma unroll
            for (int v = 0; v < V; v++) hist[j][v] = 0.f;
        }
    }
    if (off == 0) {
        const int n = last - first;
        float keep[KMAX][V];
#pragma unroll
        for (int j = 0; j < KMAX - 1; j++)
            if (j >= KMAX - K) input(n - (KMAX - 1) + j, keep[j]);
#pragma unroll
        for (int j = 0; j < KMAX - 1; j++)
            if (j >= KMAX - K)
#pragma unroll
                for (int v = 0; v < V; v++) st[(size_t)(j - (KMAX - K)) * channels + v] = keep[j][v];
    }
    constexpr int GROUP = 4;  // tokens requested together
    for (int tg = t0; tg < t1; tg += GROUP) {
        Pack<T, V> in[GROUP];
#pragma unroll
        for (int k = 0; k < GROUP; k++) in[k] = *reinterpret_cast<const Pack<T, V>*>(x + (size_t)min(tg + k, t1 - 1) * x_stride + c);
#pragma unroll
        for (int k = 0; k < GROUP; k++) {
            if (tg + k < t1) {
                Pack<T, V> o;
#pragma unroll
                for (int v = 0; v < V; v++) {
                    const float xv = to_f32(in[k].v[v]);
                    float acc = fmaf(xv, tap[KMAX - 1][v], b[v]);
#pragma unroll
                    for (int j = 0; j < KMAX - 1; j++) acc = fmaf(hist[j][v], tap[j][v], acc);
#pragma unroll
                    for (int j = 0; j < KMAX - 2; j++) hist[j][v] = hist[j + 1][v];
                    if (KMAX > 1) hist[KMAX > 1 ? KMAX - 2 : 0][v] = xv;
                    o.v[v] = from_f32<T>(silu_for<T>(acc));
                }
                *reinterpret_cast<Pack<T, V>*>(out + (size_t)(tg + k) * channels + c) = o;
            }
        }
    }
}

// ---- selective scan ---------------------------------------------------------------------------------------------
struct ScanParams {
    void* y;                 // [T, C]
    const void* x;           // [T, C]
    const void* z;           // gate, row stride z_stride
    int64_t z_stride;
    const float* dt;         // [T, C] before bias and softplus
    const float* dt_bias;    // [C]
    const float* A;          // [C, N] (negative)
    const float* bc;         // row t: B at bc + t * bc_stride, C behind it
    int64_t bc_stride;
    const float* D;          // [C]
    float* state;            // [slots, C, N]
    float* piece_state;      // [pieces, C, N]
    float* piece_dt;         // [pieces, C]: sum of dt over the piece
    int C, N;
    int run;                 // pieces a CTA takes (0: whole spans)
    ca_spans sp;
};
constexpr int SCAN_THREADS = 128;
constexpr int SCAN_TOKENS = 32;  // tokens whose B and C are staged at a time (two buffers)


// L lanes share a channel, NS states each.  Of a group of tokens, lane i of a channel reads the inputs of tokens i, i + L,
// ... and evaluates their step size and, at the end, their output; dt and dt x travel by shuffles.
// PHASE 0: whole spans: state in, outputs, state out (spans in turn per CTA column).  1: end state of the run from zero, and
// sum of dt.  2: outputs from the run's initial state.
template <typename T, int L, int NS, int PHASE>
__global__ void __launch_bounds__(SCAN_THREADS, 8) scan_kernel(const ScanParams p) {
    extern __shared__ __align__(16) float bc_s[];  // 2 x [SCAN_TOKENS][B: L * NS | C: L * NS], zero past N
    constexpr int GROUP = L <= 8 ? 8 : L;  // tokens whose x, dt, z are requested together, one group ahead
    constexpr int NP = L * NS, OWN = (GROUP + L - 1) / L, BUF = SCAN_TOKENS * 2 * NP;
    const int c = blockIdx.x * (SCAN_THREADS / L) + threadIdx.x / L;
    const int ln = threadIdx.x & (L - 1), base = (threadIdx.x & 31) & ~(L - 1), n0 = ln * NS, N = p.N;
    const bool on = c < p.C;
    const int cc = on ? c : p.C - 1;
    uint64_t A2[NS / 2];  // pairs of states
#pragma unroll
    for (int i = 0; i < NS; i += 2) {
        const float* a = p.A + (size_t)cc * N + n0 + i;
        A2[i / 2] = pair_f32(n0 + i < N ? a[0] * LOG2E : 0.f, n0 + i + 1 < N ? a[1] * LOG2E : 0.f);
    }
    const float bias = p.dt_bias[cc], D = PHASE == 1 ? 0.f : p.D[cc];
    const T* X = static_cast<const T*>(p.x) + cc;
    const T* Z = static_cast<const T*>(p.z) + cc;
    T* Y = static_cast<T*>(p.y) + cc;
    const float* DT = p.dt + cc;
    // the padding past N is never copied into
    for (int i = threadIdx.x; i < 2 * BUF; i += SCAN_THREADS)
        if (i % NP >= N) bc_s[i] = 0.f;
    for (int unit = blockIdx.y; unit < (PHASE == 0 ? p.sp.n_entries : p.sp.n_work); unit += gridDim.y) {
        int e = unit, t0, t1;
        if (PHASE == 0) {
            t0 = p.sp.cu[e];
            t1 = p.sp.cu[e + 1];
        } else {
            const int4 wk = reinterpret_cast<const int4*>(p.sp.work)[unit];
            if (wk.w % p.run) continue;  // a run starts at every run-th piece
            e = wk.x;
            t0 = wk.y;
            t1 = min(p.sp.cu[e + 1], t0 + p.run * p.sp.work_len);
        }
        float S[NS];
        float* slot = p.state + ((size_t)p.sp.slot[e] * p.C + cc) * N + n0;
        float* piece = PHASE == 0 ? nullptr : p.piece_state + ((size_t)unit * p.C + cc) * N + n0;
        const bool live = p.sp.start[e] > 0;
        const bool vec = N % 4 == 0;
        const float* from = PHASE == 0 ? slot : piece;
#pragma unroll
        for (int i = 0; i < NS; i++) S[i] = 0.f;
        if (PHASE == 2 || (PHASE == 0 && live)) {
            if (vec) {
#pragma unroll
                for (int i = 0; i < NS; i += 4)
                    if (n0 + i < N) {
                        const float4 v = *reinterpret_cast<const float4*>(from + i);
                        S[i] = v.x; S[i + 1] = v.y; S[i + 2] = v.z; S[i + 3] = v.w;
                    }
            } else {
#pragma unroll
                for (int i = 0; i < NS; i++)
                    if (n0 + i < N) S[i] = from[i];
            }
        }
        uint64_t S2[NS / 2];
#pragma unroll
        for (int i = 0; i < NS; i += 2) S2[i / 2] = pair_f32(S[i], S[i + 1]);
        float sum_dt = 0.f;
        auto stage = [&](int tb, int buf) {  // B and C of the next tokens, asynchronously
            const int nt = min(SCAN_TOKENS, t1 - tb);
            for (int i = threadIdx.x; i < nt * 2 * N; i += SCAN_THREADS) {
                const int tt = i / (2 * N), r = i - tt * 2 * N;
                const uint32_t dst = (uint32_t)__cvta_generic_to_shared(bc_s + buf * BUF + tt * 2 * NP + (r < N ? r : r - N + NP));
                asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(p.bc + (size_t)(tb + tt) * p.bc_stride + r) : "memory");
            }
        };
        float xs[OWN], ds[OWN], zs[OWN], nd[OWN];
        T nx[OWN], nz[OWN];  // as they come: a conversion here would wait for the loads
        auto request = [&](int t) {  // this lane's tokens of the group that starts at t
#pragma unroll
            for (int k = 0; k < OWN; k++) {
                const int tk = ln + k * L;
                nd[k] = 0.f;
                nx[k] = nz[k] = from_f32<T>(0.f);
                if (tk < GROUP && t + tk < t1) {
                    nx[k] = X[(size_t)(t + tk) * p.C];
                    nd[k] = DT[(size_t)(t + tk) * p.C];
                    if (PHASE != 1) nz[k] = Z[(size_t)(t + tk) * p.z_stride];
                }
            }
        };
        __syncthreads();  // nobody reads the buffers of the span before any more
        stage(t0, 0);
        asm volatile("cp.async.commit_group;" ::: "memory");
        request(t0);
        int buf = 0;
        for (int tb = t0; tb < t1; tb += SCAN_TOKENS, buf ^= 1) {
            const int nt = min(SCAN_TOKENS, t1 - tb);
            if (tb > t0) __syncthreads();  // the other buffer is free
            if (tb + SCAN_TOKENS < t1) stage(tb + SCAN_TOKENS, buf ^ 1);
            asm volatile("cp.async.commit_group;" ::: "memory");
            asm volatile("cp.async.wait_group 1;" ::: "memory");
            __syncthreads();
            for (int g = 0; g < nt; g += GROUP) {
                float us[OWN], ys[OWN];
#pragma unroll
                for (int k = 0; k < OWN; k++) {
                    xs[k] = to_f32(nx[k]);
                    zs[k] = to_f32(nz[k]);
                    ds[k] = softplus_f(nd[k] + bias);
                    us[k] = ds[k] * xs[k];
                    ys[k] = 0.f;
                }
                if (tb + g + GROUP < t1) request(tb + g + GROUP);
                auto token = [&](int k) {
                    const int own = k % L;
                    float dt = ds[k / L], u = us[k / L];
                    if (L > 1) {
                        dt = __shfl_sync(0xffffffffu, dt, base + own);
                        u = __shfl_sync(0xffffffffu, u, base + own);
                    }
                    const float* B = bc_s + buf * BUF + (g + k) * 2 * NP + n0;
                    const uint64_t dt2 = pair_f32(dt, dt), u2 = pair_f32(u, u);
                    uint64_t y2 = 0;
#pragma unroll
                    for (int i = 0; i < NS; i += 4) {
                        const ulonglong2 b4 = *reinterpret_cast<const ulonglong2*>(B + i), c4 = *reinterpret_cast<const ulonglong2*>(B + NP + i);
                        const uint64_t bb[2] = {b4.x, b4.y}, cc2[2] = {c4.x, c4.y};
#pragma unroll
                        for (int j = 0; j < 2; j++) {
                            uint64_t& s2 = S2[i / 2 + j];
                            float lo, hi;
                            unpair_f32(mul_f32x2(dt2, A2[i / 2 + j]), lo, hi);
                            s2 = fma_f32x2(pair_f32(exp2_approx(lo), exp2_approx(hi)), s2, mul_f32x2(u2, bb[j]));
                            if (PHASE != 1) y2 = fma_f32x2(s2, cc2[j], y2);
                        }
                    }
                    float y, y_hi;
                    unpair_f32(y2, y, y_hi);
                    y += y_hi;
                    if (PHASE == 1) {
                        sum_dt += dt;
                    } else {
#pragma unroll
                        for (int off = L >> 1; off >= 1; off >>= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
                        if (own == ln) ys[k / L] = y;
                    }
                };
                if (nt - g >= GROUP) {
#pragma unroll
                    for (int k = 0; k < GROUP; k++) token(k);
                } else {
#pragma unroll
                    for (int k = 0; k < GROUP; k++)
                        if (g + k < nt) token(k);
                }
                if (PHASE != 1) {
#pragma unroll
                    for (int k = 0; k < OWN; k++) {
                        const int tk = ln + k * L;
                        if (on && tk < GROUP && g + tk < nt)
                            Y[(size_t)(tb + g + tk) * p.C] = from_f32<T>(fmaf(D, xs[k], ys[k]) * silu_for<T>(zs[k]));
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < NS; i += 2) unpair_f32(S2[i / 2], S[i], S[i + 1]);
        if (PHASE != 2 && on) {
            float* dst = PHASE == 0 ? slot : piece;
            if (vec) {
#pragma unroll
                for (int i = 0; i < NS; i += 4)
                    if (n0 + i < N) *reinterpret_cast<float4*>(dst + i) = make_float4(S[i], S[i + 1], S[i + 2], S[i + 3]);
            } else {
#pragma unroll
                for (int i = 0; i < NS; i++)
                    if (n0 + i < N) dst[i] = S[i];
            }
            if (PHASE == 1 && ln == 0) p.piece_dt[(size_t)unit * p.C + c] = sum_dt;
        }
    }
}

// One token per span: four states per lane straight from and to memory, a few spans in turn per CTA so that A is read
// once for them, everything of the next span requested before this one is worked on.
template <typename T, int L, bool VEC>
__global__ void __launch_bounds__(SCAN_THREADS) scan_step_kernel(const ScanParams p) {
    const int c = blockIdx.x * (SCAN_THREADS / L) + threadIdx.x / L;
    const int ln = threadIdx.x & (L - 1), N = p.N;
    const bool on = c < p.C;
    const int cc = on ? c : p.C - 1;
    constexpr int NS = 4;
    const int n0 = ln * NS;
    float A2[NS];
#pragma unroll
    for (int i = 0; i < NS; i++) A2[i] = n0 + i < N ? p.A[(size_t)cc * N + n0 + i] * LOG2E : 0.f;
    const float bias = p.dt_bias[cc], D = p.D[cc];
    struct Inputs {  // of one span, as they come
        float S[NS], B[NS], C[NS], dt;
        T x, z;
    } in;
    auto request = [&](int e) {
#pragma unroll
        for (int i = 0; i < NS; i++) in.S[i] = in.B[i] = in.C[i] = 0.f;
        if (e >= p.sp.n_entries) return;
        const size_t t = p.sp.cu[e];
        in.x = static_cast<const T*>(p.x)[t * p.C + cc];
        in.z = static_cast<const T*>(p.z)[t * p.z_stride + cc];
        in.dt = p.dt[t * p.C + cc];
        const float* B = p.bc + t * p.bc_stride + n0;
#pragma unroll
        for (int i = 0; i < NS; i++)
            if (n0 + i < N) {
                in.B[i] = __ldg(B + i);
                in.C[i] = __ldg(B + N + i);
            }
        if (p.sp.start[e] == 0) return;
        const float* s = p.state + ((size_t)p.sp.slot[e] * p.C + cc) * N + n0;
        if (VEC) {
            if (n0 < N) {
                const float4 v = *reinterpret_cast<const float4*>(s);
                in.S[0] = v.x; in.S[1] = v.y; in.S[2] = v.z; in.S[3] = v.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < NS; i++)
                if (n0 + i < N) in.S[i] = s[i];
        }
    };
    request(blockIdx.y);
    for (int e = blockIdx.y; e < p.sp.n_entries; e += gridDim.y) {
        Inputs now = in;
        request(e + gridDim.y);
        const float x = to_f32(now.x), dt = softplus_f(now.dt + bias), u = dt * x;
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NS; i++) {
            now.S[i] = fmaf(exp2_approx(dt * A2[i]), now.S[i], u * now.B[i]);
            y = fmaf(now.S[i], now.C[i], y);
        }
#pragma unroll
        for (int off = L >> 1; off >= 1; off >>= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
        float* s = p.state + ((size_t)p.sp.slot[e] * p.C + cc) * N + n0;
        if (on) {
            if (VEC) {
                if (n0 < N) *reinterpret_cast<float4*>(s) = make_float4(now.S[0], now.S[1], now.S[2], now.S[3]);
            } else {
#pragma unroll
                for (int i = 0; i < NS; i++)
                    if (n0 + i < N) s[i] = now.S[i];
            }
            if (ln == 0) static_cast<T*>(p.y)[(size_t)p.sp.cu[e] * p.C + c] = from_f32<T>(fmaf(D, x, y) * silu_for<T>(to_f32(now.z)));
        }
    }
}

// per (span, channel, state): end states of the runs -> initial states, and the span's end state to its slot
__global__ void scan_sweep_kernel(const ScanParams p) {
    const int e = blockIdx.y;
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x, CN = (int64_t)p.C * p.N;
    if (i >= CN) return;
    const int c = (int)(i / p.N);
    const float A2 = p.A[i] * LOG2E;
    float* slot = p.state + (size_t)p.sp.slot[e] * CN + i;
    float S = p.sp.start[e] > 0 ? *slot : 0.f;
    for (int w = p.sp.work_off[e]; w < p.sp.work_off[e + 1]; w += p.run) {
        float* piece = p.piece_state + (size_t)w * CN + i;
        const float local = *piece;
        *piece = S;
        S = fmaf(exp2_approx(A2 * p.piece_dt[(size_t)w * p.C + c]), S, local);
    }
    *slot = S;
}

// Lanes per channel: eight states each in the scan, whose inner loop then is bound by the exponentials and not by shuffles
// and shared memory; four in the decode step, where the state's way through memory is what counts.
int scan_lanes(int n_states, int per_lane) {
    int lanes = 1;
    while (lanes < 32 && lanes * per_lane < n_states) lanes *= 2;
    return lanes;
}
// Pieces per CTA.  Sequential over whole spans (0) when spans and channels alone fill the GPU; else runs that do.
int scan_run(const ca_spans& sp, int channels, int n_states) {
    const int per_block = SCAN_THREADS / scan_lanes(n_states, 8);
    const int64_t blocks = (channels + per_block - 1) / per_block;
    if (sp.n_work == sp.n_entries || blocks * sp.n_entries >= 444) return 0;
    const int64_t run = (blocks * sp.n_work + 148 * 7 - 1) / (148 * 7);  // one wave of about seven CTAs per SM
    const int longest = (sp.max_tokens + sp.work_len - 1) / sp.work_len;
    return run >= longest ? 0 : (int)run;
}

template <typename T, int L>
void launch_scan(const ScanParams& p, cudaStream_t stream) {
    constexpr int NS = 8, per_block = SCAN_THREADS / L;
    const int blocks = (p.C + per_block - 1) / per_block;
    const size_t smem = (size_t)2 * SCAN_TOKENS * 2 * L * NS * sizeof(float);  // at most 128 KiB (256 states)
    if (smem > 48 * 1024) {
        cudaFuncSetAttribute(scan_kernel<T, L, NS, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cudaFuncSetAttribute(scan_kernel<T, L, NS, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        cudaFuncSetAttribute(scan_kernel<T, L, NS, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    }
    if (p.run == 0) {
        scan_kernel<T, L, NS, 0><<<dim3(blocks, p.sp.n_entries), SCAN_THREADS, smem, stream>>>(p);
    } else {
        scan_kernel<T, L, NS, 1><<<dim3(blocks, p.sp.n_work), SCAN_THREADS, smem, stream>>>(p);
        scan_sweep_kernel<<<dim3((unsigned)(((int64_t)p.C * p.N + 255) / 256), p.sp.n_entries), 256, 0, stream>>>(p);
        scan_kernel<T, L, NS, 2><<<dim3(blocks, p.sp.n_work), SCAN_THREADS, smem, stream>>>(p);
    }
}
template <typename T, int L>
void launch_scan_step(const ScanParams& p, cudaStream_t stream) {
    constexpr int per_block = SCAN_THREADS / L;
    const int blocks = (p.C + per_block - 1) / per_block;
    const dim3 grid(blocks, std::min(p.sp.n_entries, std::max(1, 148 * 64 / blocks)));
    if (p.N % 4 == 0) scan_step_kernel<T, L, true><<<grid, SCAN_THREADS, 0, stream>>>(p);
    else scan_step_kernel<T, L, false><<<grid, SCAN_THREADS, 0, stream>>>(p);
}
// f(integral_constant L)
template <typename F> void by_lanes(int lanes, F&& f) {
    switch (lanes) {
        case 1: f(std::integral_constant<int, 1>()); break;
        case 2: f(std::integral_constant<int, 2>()); break;
        case 4: f(std::integral_constant<int, 4>()); break;
        case 8: f(std::integral_constant<int, 8>()); break;
        case 16: f(std::integral_constant<int, 16>()); break;
        default: f(std::integral_constant<int, 32>());
    }
}

// ---- linear attention with decay --------------------------------------------------------------------------------
struct DecayParams {
    void* out;               // [T, H * dv]
    const void* qkv;         // row t: q heads | k heads | v heads, before SiLU
    int64_t row_stride;
    const float* decay;      // [H]
    float* state;            // [slots, H, dk, dv]
    float* scratch;          // [pieces, H, dk, dv] or null
    int H, dk, dv;
    ca_spans sp;
};

// One token per span: CTA per (span, head).  Threads span the columns of the state (VEC wide) and split its rows.
constexpr int DECAY_STEP_THREADS = 256;
template <typename T, int V>
__global__ void __launch_bounds__(DECAY_STEP_THREADS) decay_step_kernel(const DecayParams p) {
    extern __shared__ float sm[];
    float* q = sm;                       // [dk]
    float* k = q + p.dk;                 // [dk]
    float* red = k + p.dk;               // [row groups][dv]
    const int e = blockIdx.y, h = blockIdx.x, t = p.sp.cu[e];
    const T* row = static_cast<const T*>(p.qkv) + (size_t)t * p.row_stride;
    const int Hk = p.H * p.dk;
    for (int i = threadIdx.x; i < p.dk; i += blockDim.x) {
        q[i] = silu_f(to_f32(row[h * p.dk + i]));
        k[i] = silu_f(to_f32(row[Hk + h * p.dk + i]));
    }
    __syncthreads();
    const int cols = p.dv / V, groups = max(1, DECAY_STEP_THREADS / cols);
    const float d = p.decay[h];
    const bool live = p.sp.start[e] > 0;
    float* S = p.state + ((size_t)p.sp.slot[e] * p.H + h) * p.dk * p.dv;
    // a group of `cols` threads takes every groups-th row; wider values than threads loop over the columns
    for (int base = 0; base < cols; base += DECAY_STEP_THREADS) {
        const int cg = cols <= DECAY_STEP_THREADS ? threadIdx.x % cols : base + threadIdx.x;
        const int rg = cols <= DECAY_STEP_THREADS ? threadIdx.x / cols : 0;
        if (rg < groups && cg < cols) {
            float v[V], acc[V];
#pragma unroll
            for (int i = 0; i < V; i++) {
                v[i] = silu_f(to_f32(row[2 * Hk + h * p.dv + cg * V + i]));
                acc[i] = 0.f;
            }
            constexpr int AHEAD = 8;  // rows requested together
            for (int r0 = rg; r0 < p.dk; r0 += AHEAD * groups) {
                Pack<float, V> s[AHEAD];
#pragma unroll
                for (int x = 0; x < AHEAD; x++) {
                    const int r = r0 + x * groups;
                    if (live && r < p.dk) {
                        s[x] = *reinterpret_cast<const Pack<float, V>*>(S + (size_t)r * p.dv + cg * V);
                    } else {
#pragma unroll
                        for (int i = 0; i < V; i++) s[x].v[i] = 0.f;
                    }
                }
#pragma unroll
                for (int x = 0; x < AHEAD; x++) {
                    const int r = r0 + x * groups;
                    if (r >= p.dk) break;
#pragma unroll
                    for (int i = 0; i < V; i++) {
                        s[x].v[i] = fmaf(k[r], v[i], d * s[x].v[i]);
                        acc[i] = fmaf(q[r], s[x].v[i], acc[i]);
                    }
                    *reinterpret_cast<Pack<float, V>*>(S + (size_t)r * p.dv + cg * V) = s[x];
                }
            }
#pragma unroll
            for (int i = 0; i < V; i++) red[rg * p.dv + cg * V + i] = acc[i];
        }
    }
    __syncthreads();
    T* out = static_cast<T*>(p.out) + ((size_t)t * p.H + h) * p.dv;
    for (int i = threadIdx.x; i < p.dv; i += blockDim.x) {
        float s = 0.f;
        for (int r = 0; r < min(groups, p.dk); r++) s += red[r * p.dv + i];
        out[i] = from_f32<T>(s);
    }
}

// Whole spans, fp32 on CUDA cores: CTA per (span, head, 32 columns of the values), blocks of 32 tokens in turn.
constexpr int DS_TOK = 32, DS_COL = 32, DS_THREADS = 256;
template <typename T>
__global__ void __launch_bounds__(DS_THREADS) decay_span_kernel(const DecayParams p) {
    extern __shared__ float sm[];
    const int dk = p.dk, pitch = dk + 1;
    float* q = sm;                              // [32][dk + 1]
    float* k = q + DS_TOK * pitch;              // [32][dk + 1]
    float* S = k + DS_TOK * pitch;              // [dk][33]
    float* v = S + dk * (DS_COL + 1);           // [32][33]
    float* P = v + DS_TOK * (DS_COL + 1);       // [32][33]
    float* pw = P + DS_TOK * (DS_COL + 1);      // decay^0 .. decay^32
    const int h = blockIdx.x, c0 = blockIdx.y * DS_COL, e = blockIdx.z;
    const int n_cols = min(DS_COL, p.dv - c0), Hk = p.H * dk;
    const float d = p.decay[h];
    for (int i = threadIdx.x; i <= DS_TOK; i += DS_THREADS) pw[i] = powf(d, (float)i);
    float* St = p.state + ((size_t)p.sp.slot[e] * p.H + h) * dk * p.dv;
    const bool live = p.sp.start[e] > 0;
    for (int i = threadIdx.x; i < dk * DS_COL; i += DS_THREADS) {
        const int r = i / DS_COL, c = i % DS_COL;
        S[r * (DS_COL + 1) + c] = live && c < n_cols ? St[(size_t)r * p.dv + c0 + c] : 0.f;
    }
    const int t_end = p.sp.cu[e + 1];
    for (int t0 = p.sp.cu[e]; t0 < t_end; t0 += DS_TOK) {
        const int n = min(DS_TOK, t_end - t0);
        __syncthreads();
        for (int i = threadIdx.x; i < DS_TOK * dk; i += DS_THREADS) {
            const int r = i / dk, c = i % dk;
            const T* row = static_cast<const T*>(p.qkv) + (size_t)(t0 + min(r, n - 1)) * p.row_stride;
            q[r * pitch + c] = r < n ? silu_f(to_f32(row[h * dk + c])) : 0.f;
            k[r * pitch + c] = r < n ? silu_f(to_f32(row[Hk + h * dk + c])) : 0.f;
        }
        for (int i = threadIdx.x; i < DS_TOK * DS_COL; i += DS_THREADS) {
            const int r = i / DS_COL, c = i % DS_COL;
            const T* row = static_cast<const T*>(p.qkv) + (size_t)(t0 + min(r, n - 1)) * p.row_stride;
            v[r * (DS_COL + 1) + c] = r < n && c < n_cols ? silu_f(to_f32(row[2 * Hk + h * p.dv + c0 + c])) : 0.f;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < DS_TOK * DS_TOK; i += DS_THREADS) {
            const int r = i / DS_TOK, j = i % DS_TOK;
            float acc = 0.f;
            if (j <= r) {
                for (int x = 0; x < dk; x++) acc = fmaf(q[r * pitch + x], k[j * pitch + x], acc);
                acc *= pw[r - j];
            }
            P[r * (DS_COL + 1) + j] = acc;
        }
        __syncthreads();
        for (int i = threadIdx.x; i < DS_TOK * DS_COL; i += DS_THREADS) {
            const int r = i / DS_COL, c = i % DS_COL;
            if (r >= n || c >= n_cols) continue;
            float far = 0.f, near = 0.f;
            for (int x = 0; x < dk; x++) far = fmaf(q[r * pitch + x], S[x * (DS_COL + 1) + c], far);
            for (int j = 0; j <= r; j++) near = fmaf(P[r * (DS_COL + 1) + j], v[j * (DS_COL + 1) + c], near);
            static_cast<T*>(p.out)[((size_t)(t0 + r) * p.H + h) * p.dv + c0 + c] = from_f32<T>(fmaf(pw[r + 1], far, near));
        }
        __syncthreads();
        for (int i = threadIdx.x; i < dk * DS_COL; i += DS_THREADS) {
            const int r = i / DS_COL, c = i % DS_COL;
            float acc = pw[n] * S[r * (DS_COL + 1) + c];
            for (int j = 0; j < n; j++) acc = fmaf(pw[n - 1 - j] * k[j * pitch + r], v[j * (DS_COL + 1) + c], acc);
            S[r * (DS_COL + 1) + c] = acc;
        }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < dk * DS_COL; i += DS_THREADS) {
        const int r = i / DS_COL, c = i % DS_COL;
        if (c < n_cols) St[(size_t)r * p.dv + c0 + c] = S[r * (DS_COL + 1) + c];
    }
}

bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }

template <typename T>
int conv_silu(void* out, const void* x, int64_t x_stride, const float* taps, const float* bias, float* state, const ca_spans& sp,
              int channels, int K, cudaStream_t stream) {
    auto packs = [&](int v) { return channels % v == 0 && x_stride % v == 0 && reinterpret_cast<uintptr_t>(x) % (v * sizeof(T)) == 0; };
    const int v = packs(4) && K <= 4 ? 4 : (packs(2) ? 2 : 1);
    const int per = 128 * v;
    const dim3 grid((channels + per - 1) / per, sp.n_work);
    T* o = static_cast<T*>(out);
    const T* in = static_cast<const T*>(x);
#define CA_CONV(V, KM) conv_silu_kernel<T, V, KM><<<grid, 128, 0, stream>>>(o, in, x_stride, taps, bias, state, sp, channels, K)
    if (v == 4) {
        CA_CONV(4, 4);
    } else if (v == 2) {
        if (K <= 4) CA_CONV(2, 4); else CA_CONV(2, 16);
    } else {
        if (K <= 4) CA_CONV(1, 4); else CA_CONV(1, 16);
    }
#undef CA_CONV
    return done();
}

template <typename T>
int selective_scan(const ScanParams& p, cudaStream_t stream) {
    if (p.sp.max_tokens == 1 && p.N <= 128)
        by_lanes(scan_lanes(p.N, 4), [&](auto l) { launch_scan_step<T, decltype(l)::value>(p, stream); });
    else
        by_lanes(scan_lanes(p.N, 8), [&](auto l) { launch_scan<T, decltype(l)::value>(p, stream); });
    return done();
}

// Pieces per CTA of the tensor-core kernels (one CTA per SM; an even number, for blocks of 128 tokens): the run length that needs the fewest block times, counting two
// passes for runs and one for whole spans (0).
int decay_run(const ca_spans& sp, int heads) {
    const int longest = (sp.max_tokens + sp.work_len - 1) / sp.work_len;
    if (longest <= 1) return 0;
    auto waves = [](int64_t ctas) { return (double)((ctas + 147) / 148); };
    double best = waves((int64_t)sp.n_entries * heads) * longest;
    int best_run = 0;
    for (int run = 2; run < longest; run += 2) {
        const int64_t runs = (sp.n_work + (int64_t)(run - 1) * sp.n_entries) / run;  // at most
        // in times of a piece: a run's two passes with their start, and the sweep over the runs
        const double cost = waves(runs * heads) * (run + 1.0) * 1.75 + 2.0 + 0.2 * runs;
        if (cost < best) {
            best = cost;
            best_run = run;
        }
    }
    return best_run;
}

template <typename T>
int decay_attention(const DecayParams& p, cudaStream_t stream) {
    if (p.sp.max_tokens == 1) {
        const bool v4 = p.dv % 4 == 0;
        const int cols = p.dv / (v4 ? 4 : 1), groups = cols >= DECAY_STEP_THREADS ? 1 : DECAY_STEP_THREADS / cols;
        const size_t smem = (size_t)(2 * p.dk + groups * p.dv) * sizeof(float);
        const dim3 grid(p.H, p.sp.n_entries);
        if (v4) decay_step_kernel<T, 4><<<grid, DECAY_STEP_THREADS, smem, stream>>>(p);
        else decay_step_kernel<T, 1><<<grid, DECAY_STEP_THREADS, smem, stream>>>(p);
        return done();
    }
    if (std::is_same<T, __nv_bfloat16>::value && decay_mma_serves(p.dk, p.dv, p.row_stride, p.qkv, p.sp.work_len)) {
        DecayMmaParams m{p.out, p.qkv, p.row_stride, p.decay, p.state, p.scratch, p.H, p.dk, p.dv, decay_run(p.sp, p.H), p.sp};
        if (m.run > 0 && !p.scratch) return fail("decay_attention: this batch needs scratch");
        // short portions leave most of a 128-token block empty
        const bool tc = decay_tc_serves(p.dk, p.dv) && p.sp.max_tokens > 32;
        const cudaError_t e = tc ? launch_decay_tc(m, stream) : launch_decay_mma(m, stream);
        return e == cudaSuccess ? CA_OK : fail(cudaGetErrorString(e), CA_ERR_CUDA);
    }
    const size_t smem = (size_t)(2 * DS_TOK * (p.dk + 1) + p.dk * (DS_COL + 1) + 2 * DS_TOK * (DS_COL + 1) + DS_TOK + 1) * sizeof(float);
    const cudaError_t e = cudaFuncSetAttribute(decay_span_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(cudaGetErrorString(e), CA_ERR_CUDA);
    const dim3 grid(p.H, (p.dv + DS_COL - 1) / DS_COL, p.sp.n_entries);
    decay_span_kernel<T><<<grid, DS_THREADS, smem, stream>>>(p);
    return done();
}

bool spans_ok(const ca_spans* sp) {
    return sp && sp->n_entries > 0 && sp->n_tokens >= sp->n_entries && sp->n_work >= sp->n_entries && sp->cu && sp->start &&
           sp->slot && sp->work && sp->work_off && aligned16(sp->work);
}

}  // namespace
}  // namespace ca

using namespace ca;

extern "C" {

int ca_conv_silu(void* out, const void* x, int64_t x_stride, const float* taps, const float* bias, float* state, const ca_spans* sp,
                 int channels, int n_taps, int dtype, ca_stream stream) {
    if (!spans_ok(sp)) return fail("conv_silu: bad spans");
    if (channels <= 0 || n_taps < 1 || n_taps > 16 || n_taps > sp->work_len) return fail("conv_silu: 1 to 16 taps, no more than a piece has tokens");
    if (!out || !x || !taps || !bias || !state) return fail("conv_silu: null pointer");
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == CA_DTYPE_BF16) return conv_silu<__nv_bfloat16>(out, x, x_stride, taps, bias, state, *sp, channels, n_taps, s);
    if (dtype == CA_DTYPE_F32) return conv_silu<float>(out, x, x_stride, taps, bias, state, *sp, channels, n_taps, s);
    return fail("conv_silu: unknown element type");
}

int64_t ca_scan_scratch_floats(const ca_spans* sp, int channels, int n_states) {
    if (!sp || channels <= 0 || n_states <= 0 || scan_run(*sp, channels, n_states) == 0) return 0;
    return (int64_t)sp->n_work * channels * ((int64_t)n_states + 1);
}

int ca_selective_scan(void* y, const void* x, const void* z, int64_t z_stride, const float* dt, const float* dt_bias, const float* A,
                      const float* bc, int64_t bc_stride, const float* D, float* state, float* scratch, const ca_spans* sp,
                      int channels, int n_states, int dtype, ca_stream stream) {
    if (!spans_ok(sp)) return fail("selective_scan: bad spans");
    if (channels <= 0 || n_states < 1 || n_states > 256) return fail("selective_scan: 1 to 256 states per channel");
    if (!y || !x || !z || !dt || !dt_bias || !A || !bc || !D || !state) return fail("selective_scan: null pointer");
    ScanParams p;
    p.run = scan_run(*sp, channels, n_states);
    if (p.run > 0 && !scratch) return fail("selective_scan: this batch needs scratch");
    p.y = y; p.x = x; p.z = z; p.z_stride = z_stride; p.dt = dt; p.dt_bias = dt_bias; p.A = A; p.bc = bc; p.bc_stride = bc_stride;
    p.D = D; p.state = state; p.piece_state = scratch;
    p.piece_dt = scratch ? scratch + (size_t)sp->n_work * channels * n_states : nullptr;
    p.C = channels; p.N = n_states; p.sp = *sp;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == CA_DTYPE_BF16) return selective_scan<__nv_bfloat16>(p, s);
    if (dtype == CA_DTYPE_F32) return selective_scan<float>(p, s);
    return fail("selective_scan: unknown element type");
}

int ca_block_status(int32_t* status, ca_stream stream) {
    if (!status) return fail("block_status: null pointer");
    const cudaError_t e = read_decay_status(status, static_cast<cudaStream_t>(stream));
    return e == cudaSuccess ? CA_OK : fail(cudaGetErrorString(e), CA_ERR_CUDA);
}

int64_t ca_decay_scratch_floats(const ca_spans* sp, int n_heads, int d_key, int d_value, int dtype) {
    if (!sp || dtype != CA_DTYPE_BF16 || sp->max_tokens <= 1 || n_heads <= 0 || decay_run(*sp, n_heads) == 0) return 0;
    return (int64_t)sp->n_work * n_heads * d_key * d_value;
}

int ca_decay_attention(void* out, const void* qkv, int64_t row_stride, const float* decay, float* state, float* scratch, const ca_spans* sp,
                       int n_heads, int d_key, int d_value, int dtype, ca_stream stream) {
    if (!spans_ok(sp)) return fail("decay_attention: bad spans");
    if (n_heads <= 0 || d_key <= 0 || d_key > 256 || d_value <= 0 || d_value > 1024) return fail("decay_attention: head sizes out of range");
    if (!out || !qkv || !decay || !state) return fail("decay_attention: null pointer");
    DecayParams p;
    p.out = out; p.qkv = qkv; p.row_stride = row_stride; p.decay = decay; p.state = state; p.scratch = scratch;
    p.H = n_heads; p.dk = d_key; p.dv = d_value; p.sp = *sp;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == CA_DTYPE_BF16) return decay_attention<__nv_bfloat16>(p, s);
    if (dtype == CA_DTYPE_F32) return decay_attention<float>(p, s);
    return fail("decay_attention: unknown element type");
}

}  // extern "C"
