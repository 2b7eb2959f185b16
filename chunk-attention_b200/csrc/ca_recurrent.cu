// Recurrent sequence mixers over batches of spans (consecutive tokens of several sequences, each with a state slot):
// causal depthwise convolution + SiLU, the selective scan of Mamba, and linear attention with a per-head decay.
// States are fp32, live in [slots][...] arrays of the caller, and are read at a span's start (taken as zero at position
// 0, so a slot needs no clearing before it is used again) and written at its end.
//
// The work of a step is listed as PIECES of at most `work_len` tokens of one span (ca_spans).  A step whose spans are
// all single pieces runs a recurrence in one launch; otherwise the scan takes three: local end state of every piece
// from zero, a sweep over the pieces of each sequence that turns them into initial states, and the outputs.
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
    for (int t = t0; t < t1; t++) {
        const Pack<T, V> a = *reinterpret_cast<const Pack<T, V>*>(x + (size_t)t * x_stride + c);
        Pack<T, V> o;
#pragma unroll
        for (int v = 0; v < V; v++) {
            const float xv = to_f32(a.v[v]);
            float acc = fmaf(xv, tap[KMAX - 1][v], b[v]);
#pragma unroll
            for (int j = 0; j < KMAX - 1; j++) acc = fmaf(hist[j][v], tap[j][v], acc);
#pragma unroll
            for (int j = 0; j < KMAX - 2; j++) hist[j][v] = hist[j + 1][v];
            if (KMAX > 1) hist[KMAX > 1 ? KMAX - 2 : 0][v] = xv;
            o.v[v] = from_f32<T>(silu_f(acc));
        }
        *reinterpret_cast<Pack<T, V>*>(out + (size_t)t * channels + c) = o;
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
    int C, N, lane_shift;    // 1 << lane_shift lanes share a channel, NS states each
    ca_spans sp;
};
constexpr int SCAN_THREADS = 128;
constexpr int SCAN_TOKENS = 16;  // tokens whose B and C are staged at a time
constexpr int SCAN_GROUP = 8;    // tokens whose x, dt, z are requested together

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// PHASE 0: the span is one piece: state in, outputs, state out.  1: end state of the piece from zero, and sum of dt.
// 2: outputs from the piece's initial state.
template <typename T, int NS, int PHASE>
__global__ void __launch_bounds__(SCAN_THREADS) scan_kernel(const ScanParams p) {
    extern __shared__ float bc_s[];  // [SCAN_TOKENS][2 N]
    const int4 wk = reinterpret_cast<const int4*>(p.sp.work)[blockIdx.y];
    const int e = wk.x, t0 = wk.y, t1 = wk.z;
    const int L = 1 << p.lane_shift;
    const int c = blockIdx.x * (SCAN_THREADS >> p.lane_shift) + (threadIdx.x >> p.lane_shift);
    const int n0 = (threadIdx.x & (L - 1)) * NS, N = p.N, N2 = 2 * N;
    const bool on = c < p.C;
    const int cc = on ? c : p.C - 1;
    float S[NS], A2[NS];
    float* slot = p.state + ((size_t)p.sp.slot[e] * p.C + cc) * N;
    float* piece = p.piece_state + ((size_t)blockIdx.y * p.C + cc) * N;
    const bool live = p.sp.start[e] > 0;
#pragma unroll
    for (int i = 0; i < NS; i++) {
        const int n = n0 + i;
        A2[i] = n < N ? p.A[(size_t)cc * N + n] * LOG2E : 0.f;
        S[i] = 0.f;
        if (n < N) {
            if (PHASE == 0 && live) S[i] = slot[n];
            if (PHASE == 2) S[i] = piece[n];
        }
    }
    const float bias = p.dt_bias[cc], D = PHASE == 1 ? 0.f : p.D[cc];
    const T* X = static_cast<const T*>(p.x) + cc;
    const T* Z = static_cast<const T*>(p.z) + cc;
    T* Y = static_cast<T*>(p.y) + cc;
    const float* DT = p.dt + cc;
    float sum_dt = 0.f;
    for (int tb = t0; tb < t1; tb += SCAN_TOKENS) {
        const int nt = min(SCAN_TOKENS, t1 - tb);
        __syncthreads();
        for (int i = threadIdx.x; i < nt * N2; i += SCAN_THREADS) {
            const int tt = i / N2;
            bc_s[i] = p.bc[(size_t)(tb + tt) * p.bc_stride + (i - tt * N2)];
        }
        __syncthreads();
        for (int g = 0; g < nt; g += SCAN_GROUP) {
            float xs[SCAN_GROUP], ds[SCAN_GROUP], zs[SCAN_GROUP];
#pragma unroll
            for (int k = 0; k < SCAN_GROUP; k++) {
                const size_t t = (size_t)min(tb + g + k, t1 - 1);
                xs[k] = to_f32(X[t * p.C]);
                ds[k] = DT[t * p.C];
                if (PHASE != 1) zs[k] = to_f32(Z[t * p.z_stride]);
            }
#pragma unroll
            for (int k = 0; k < SCAN_GROUP; k++) {
                if (g + k < nt) {
                    const float dt = softplus_f(ds[k] + bias);
                    const float u = dt * xs[k];
                    const float* B = bc_s + (g + k) * N2 + n0;
                    float y = 0.f;
#pragma unroll
                    for (int i = 0; i < NS; i++) {
                        if (NS * L == N || n0 + i < N) {
                            S[i] = fmaf(exp2f(dt * A2[i]), S[i], u * B[i]);
                            if (PHASE != 1) y = fmaf(S[i], B[N + i], y);
                        }
                    }
                    if (PHASE == 1) {
                        sum_dt += dt;
                    } else {
                        for (int off = L >> 1; off >= 1; off >>= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
                        if (on && n0 == 0) Y[(size_t)(tb + g + k) * p.C] = from_f32<T>(fmaf(D, xs[k], y) * silu_f(zs[k]));
                    }
                }
            }
        }
    }
    if (!on) return;
    float* dst = PHASE == 0 ? slot : piece;
    if (PHASE != 2) {
#pragma unroll
        for (int i = 0; i < NS; i++)
            if (n0 + i < N) dst[n0 + i] = S[i];
        if (PHASE == 1 && n0 == 0) p.piece_dt[(size_t)blockIdx.y * p.C + c] = sum_dt;
    }
}

// per (span, channel, state): end states of the pieces -> initial states, and the span's end state to its slot
__global__ void scan_sweep_kernel(const ScanParams p) {
    const int e = blockIdx.y;
    const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x, CN = (int64_t)p.C * p.N;
    if (i >= CN) return;
    const int c = (int)(i / p.N);
    const float A2 = p.A[i] * LOG2E;
    float* slot = p.state + (size_t)p.sp.slot[e] * CN + i;
    float S = p.sp.start[e] > 0 ? *slot : 0.f;
    for (int w = p.sp.work_off[e]; w < p.sp.work_off[e + 1]; w++) {
        float* piece = p.piece_state + (size_t)w * CN + i;
        const float local = *piece;
        *piece = S;
        S = fmaf(exp2f(A2 * p.piece_dt[(size_t)w * p.C + c]), S, local);
    }
    *slot = S;
}

template <typename T, int NS>
void launch_scan(const ScanParams& p, int phase, cudaStream_t stream) {
    const int per_block = SCAN_THREADS >> p.lane_shift;
    const dim3 grid((p.C + per_block - 1) / per_block, p.sp.n_work);
    const size_t smem = (size_t)SCAN_TOKENS * 2 * p.N * sizeof(float);
    if (phase == 0) scan_kernel<T, NS, 0><<<grid, SCAN_THREADS, smem, stream>>>(p);
    else if (phase == 1) scan_kernel<T, NS, 1><<<grid, SCAN_THREADS, smem, stream>>>(p);
    else scan_kernel<T, NS, 2><<<grid, SCAN_THREADS, smem, stream>>>(p);
}
template <typename T>
void dispatch_scan(ScanParams& p, int phase, cudaStream_t stream) {
    // decode-like pieces: many lanes per channel, few states each (coalesced state traffic); long pieces: the fewest
    // lanes that keep a channel's states in registers
    const int max_ns = phase == 0 && p.sp.max_tokens <= 4 ? 4 : 16;
    int shift = 0;
    while (shift < 5 && (p.N + (1 << shift) - 1) / (1 << shift) > max_ns) shift++;
    const int ns = (p.N + (1 << shift) - 1) / (1 << shift);
    p.lane_shift = shift;
    if (ns <= 4) launch_scan<T, 4>(p, phase, stream);
    else if (ns <= 8) launch_scan<T, 8>(p, phase, stream);
    else if (ns <= 12) launch_scan<T, 12>(p, phase, stream);
    else launch_scan<T, 16>(p, phase, stream);
}

// ---- linear attention with decay --------------------------------------------------------------------------------
struct DecayParams {
    void* out;               // [T, H * dv]
    const void* qkv;         // row t: q heads | k heads | v heads, before SiLU
    int64_t row_stride;
    const float* decay;      // [H]
    float* state;            // [slots, H, dk, dv]
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
#pragma unroll 8
            for (int r = rg; r < p.dk; r += groups) {
                Pack<float, V>* cell = reinterpret_cast<Pack<float, V>*>(S + (size_t)r * p.dv + cg * V);
                Pack<float, V> s;
                if (live) s = *cell;
#pragma unroll
                for (int i = 0; i < V; i++) {
                    s.v[i] = fmaf(k[r], v[i], live ? d * s.v[i] : 0.f);
                    acc[i] = fmaf(q[r], s.v[i], acc[i]);
                }
                *cell = s;
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
    const bool v2 = channels % 2 == 0 && x_stride % 2 == 0 && reinterpret_cast<uintptr_t>(x) % (2 * sizeof(T)) == 0;
    const int per = 128 * (v2 ? 2 : 1);
    const dim3 grid((channels + per - 1) / per, sp.n_work);
    T* o = static_cast<T*>(out);
    const T* in = static_cast<const T*>(x);
#define CA_CONV(V, KM) conv_silu_kernel<T, V, KM><<<grid, 128, 0, stream>>>(o, in, x_stride, taps, bias, state, sp, channels, K)
    if (v2) {
        if (K <= 4) CA_CONV(2, 4); else CA_CONV(2, 16);
    } else {
        if (K <= 4) CA_CONV(1, 4); else CA_CONV(1, 16);
    }
#undef CA_CONV
    return done();
}

template <typename T>
int selective_scan(ScanParams& p, cudaStream_t stream) {
    if (p.sp.n_work == p.sp.n_entries) {
        dispatch_scan<T>(p, 0, stream);
    } else {
        dispatch_scan<T>(p, 1, stream);
        const dim3 grid((unsigned)(((int64_t)p.C * p.N + 255) / 256), p.sp.n_entries);
        scan_sweep_kernel<<<grid, 256, 0, stream>>>(p);
        dispatch_scan<T>(p, 2, stream);
    }
    return done();
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
    if (dtype == CA_DTYPE_F16) return conv_silu<__half>(out, x, x_stride, taps, bias, state, *sp, channels, n_taps, s);
    return fail("conv_silu: unknown element type");
}

int64_t ca_scan_scratch_floats(const ca_spans* sp, int channels, int n_states) {
    if (!sp || sp->n_work == sp->n_entries) return 0;
    return (int64_t)sp->n_work * channels * ((int64_t)n_states + 1);
}

int ca_selective_scan(void* y, const void* x, const void* z, int64_t z_stride, const float* dt, const float* dt_bias, const float* A,
                      const float* bc, int64_t bc_stride, const float* D, float* state, float* scratch, const ca_spans* sp,
                      int channels, int n_states, int dtype, ca_stream stream) {
    if (!spans_ok(sp)) return fail("selective_scan: bad spans");
    if (channels <= 0 || n_states < 1 || n_states > 256) return fail("selective_scan: 1 to 256 states per channel");
    if (!y || !x || !z || !dt || !dt_bias || !A || !bc || !D || !state) return fail("selective_scan: null pointer");
    if (sp->n_work != sp->n_entries && !scratch) return fail("selective_scan: spans of several pieces need scratch");
    ScanParams p;
    p.y = y; p.x = x; p.z = z; p.z_stride = z_stride; p.dt = dt; p.dt_bias = dt_bias; p.A = A; p.bc = bc; p.bc_stride = bc_stride;
    p.D = D; p.state = state; p.piece_state = scratch;
    p.piece_dt = scratch ? scratch + (size_t)sp->n_work * channels * n_states : nullptr;
    p.C = channels; p.N = n_states; p.lane_shift = 0; p.sp = *sp;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == CA_DTYPE_BF16) return selective_scan<__nv_bfloat16>(p, s);
    if (dtype == CA_DTYPE_F32) return selective_scan<float>(p, s);
    if (dtype == CA_DTYPE_F16) return selective_scan<__half>(p, s);
    return fail("selective_scan: unknown element type");
}

int ca_decay_attention(void* out, const void* qkv, int64_t row_stride, const float* decay, float* state, const ca_spans* sp,
                       int n_heads, int d_key, int d_value, int dtype, ca_stream stream) {
    if (!spans_ok(sp)) return fail("decay_attention: bad spans");
    if (n_heads <= 0 || d_key <= 0 || d_key > 256 || d_value <= 0 || d_value > 1024) return fail("decay_attention: head sizes out of range");
    if (!out || !qkv || !decay || !state) return fail("decay_attention: null pointer");
    DecayParams p;
    p.out = out; p.qkv = qkv; p.row_stride = row_stride; p.decay = decay; p.state = state;
    p.H = n_heads; p.dk = d_key; p.dv = d_value; p.sp = *sp;
    cudaStream_t s = static_cast<cudaStream_t>(stream);
    if (dtype == CA_DTYPE_BF16) return decay_attention<__nv_bfloat16>(p, s);
    if (dtype == CA_DTYPE_F32) return decay_attention<float>(p, s);
    if (dtype == CA_DTYPE_F16) return decay_attention<__half>(p, s);
    return fail("decay_attention: unknown element type");
}

}  // extern "C"
