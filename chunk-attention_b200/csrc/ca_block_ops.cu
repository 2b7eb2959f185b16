// Element-wise and row-wise kernels of decoder blocks whose residual stream is kept in fp32: token shift, gated
// sublayer output + RMS norm + residual sum, scaled residual sum + RMS norm, RMS norm of an fp32 row, gated RMS norm,
// tanh-GELU, clamped gated linear unit, soft cap of logits.  HBM / latency
// bound: one CTA per token (or a flat grid), fp32 arithmetic, 16-byte accesses where rows allow.
#include "../../include/chunk_attn_b200.h"
#include "ca_kernels.h"
#include "ca_types.cuh"

namespace ca {
namespace {

__device__ __forceinline__ float block_sum(float v) {
    __shared__ float warp_sums[32];
    v = warp_sum(v);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (lane == 0) warp_sums[warp] = v;
    __syncthreads();
    float s = lane < ((int)blockDim.x >> 5) ? warp_sums[lane] : 0.f;
    s = warp_sum(s);
    __syncthreads();
    return s;
}

template <typename T, int V> __device__ __forceinline__ void load_f(const T* p, float (&x)[V]) {
    const Pack<T, V> a = *reinterpret_cast<const Pack<T, V>*>(p);
#pragma unroll
    for (int i = 0; i < V; i++) x[i] = to_f32(a.v[i]);
}
template <typename T, int V> __device__ __forceinline__ void store_f(T* p, const float (&x)[V]) {
    Pack<T, V> a;
#pragma unroll
    for (int i = 0; i < V; i++) a.v[i] = from_f32<T>(x[i]);
    *reinterpret_cast<Pack<T, V>*>(p) = a;
}

// plain[t] = x[t] and shifted[t] = x[t] + (x[t-1] - x[t]) * mu, both rounded to T.  The row before a span's first
// token comes from the sequence's state, zeros at position 0; the thread that reads it puts the span's last row back.
template <typename T, int V>
__global__ void token_shift_kernel(const float* __restrict__ x, const float* __restrict__ mu, float* __restrict__ state,
                                   T* __restrict__ plain, T* __restrict__ shifted, const ca_spans sp, int width) {
    const int t = blockIdx.x, e = sp.entry_of[t], first = sp.cu[e];
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float h[V], prev[V], m[V];
        load_f<float, V>(x + (size_t)t * width + c, h);
        load_f<float, V>(mu + c, m);
        if (t > first) {
            load_f<float, V>(x + (size_t)(t - 1) * width + c, prev);
        } else {
            float* st = state + (size_t)sp.slot[e] * width + c;
            if (sp.start[e] > 0) {
                load_f<float, V>(st, prev);
            } else {
#pragma unroll
                for (int i = 0; i < V; i++) prev[i] = 0.f;
            }
            float last[V];
            load_f<float, V>(x + (size_t)(sp.cu[e + 1] - 1) * width + c, last);
            store_f<float, V>(st, last);
        }
        store_f<T, V>(plain + (size_t)t * width + c, h);
#pragma unroll
        for (int i = 0; i < V; i++) h[i] += (prev[i] - h[i]) * m[i];
        store_f<T, V>(shifted + (size_t)t * width + c, h);
    }
}

// g = r * sigmoid(gate + bias); x += g / rms(g) * w (in place, fp32); plain = x rounded to T.
// next_mu != null (every span has one token): also what token_shift would write for the sublayer that follows.
// A thread keeps its part of g in registers (STEPS vectors); longer rows are recomputed in the second pass.
template <typename T, int V, int STEPS>
__global__ void gated_norm_add_kernel(float* __restrict__ x, const T* __restrict__ r, int64_t r_stride, const T* __restrict__ gate,
                                      int64_t gate_stride, const float* __restrict__ bias, const float* __restrict__ w, float eps,
                                      T* __restrict__ plain, const float* __restrict__ next_mu, float* __restrict__ next_state,
                                      T* __restrict__ shifted, const ca_spans sp, int width) {
    const size_t t = blockIdx.x;
    float g[STEPS][V], xs[STEPS][V];
    float ss = 0.f;
    auto gated = [&](int c, float (&out)[V]) {
        float a[V], z[V], b[V];
        load_f<T, V>(r + t * r_stride + c, a);
        load_f<T, V>(gate + t * gate_stride + c, z);
        load_f<float, V>(bias + c, b);
#pragma unroll
        for (int i = 0; i < V; i++) out[i] = a[i] * sigmoid_for<T>(z[i] + b[i]);
    };
    const int stride = blockDim.x * V;
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) {
            load_f<float, V>(x + t * width + c, xs[s]);  // requested before the reduction
            gated(c, g[s]);
#pragma unroll
            for (int i = 0; i < V; i++) ss = fmaf(g[s][i], g[s][i], ss);
        }
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V];
        gated(c, a);
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(a[i], a[i], ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss) / width + eps);
    auto finish = [&](int c, const float (&a)[V], float (&h)[V]) {
        float ww[V];
        load_f<float, V>(w + c, ww);
#pragma unroll
        for (int i = 0; i < V; i++) h[i] += a[i] * inv * ww[i];
        store_f<float, V>(x + t * width + c, h);
        if (plain) store_f<T, V>(plain + t * width + c, h);
        if (next_mu) {
            float prev[V], m[V];
            float* st = next_state + (size_t)sp.slot[t] * width + c;
            load_f<float, V>(next_mu + c, m);
            if (sp.start[t] > 0) {
                load_f<float, V>(st, prev);
            } else {
#pragma unroll
                for (int i = 0; i < V; i++) prev[i] = 0.f;
            }
            store_f<float, V>(st, h);
#pragma unroll
            for (int i = 0; i < V; i++) h[i] += (prev[i] - h[i]) * m[i];
            store_f<T, V>(shifted + t * width + c, h);
        }
    };
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) finish(c, g[s], xs[s]);
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V], h[V];
        load_f<float, V>(x + t * width + c, h);
        gated(c, a);
        finish(c, a, h);
    }
}

// out[i] = x[row i] / rms * w, rounded to T; x may be fp32 (the residual stream) or T; with gate:
// multiplied by sigmoid(gate[i]).  rows: which rows of x (null: row i).
template <typename TI, typename T, int V>
__global__ void norm_rows_kernel(T* __restrict__ out, const TI* __restrict__ x, int64_t x_stride, const int32_t* __restrict__ rows,
                                 const float* __restrict__ w, const T* __restrict__ gate, int64_t gate_stride, float eps, int width) {
    const size_t t = blockIdx.x;
    const TI* src = x + (size_t)(rows ? rows[t] : t) * x_stride;
    constexpr int STEPS = V == 1 ? 4 : (V == 8 ? 1 : 2);  // of the row a thread keeps in registers, gate included
    float kept[STEPS][V], f[STEPS][V];  // the factor (weight and gate) is ready before the reduction
    float ss = 0.f;
    auto factor = [&](int c, float (&out)[V]) {
        load_f<float, V>(w + c, out);
        if (gate) {
            float z[V];
            load_f<T, V>(gate + t * gate_stride + c, z);
#pragma unroll
            for (int i = 0; i < V; i++) out[i] *= sigmoid_for<T>(z[i]);
        }
    };
    const int stride = blockDim.x * V;
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) {
            load_f<TI, V>(src + c, kept[s]);
            factor(c, f[s]);
#pragma unroll
            for (int i = 0; i < V; i++) ss = fmaf(kept[s][i], kept[s][i], ss);
        }
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V];
        load_f<TI, V>(src + c, a);
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(a[i], a[i], ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss) / width + eps);
    auto finish = [&](int c, float (&a)[V], const float (&ff)[V]) {
#pragma unroll
        for (int i = 0; i < V; i++) a[i] *= inv * ff[i];
        store_f<T, V>(out + t * width + c, a);
    };
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) finish(c, kept[s], f[s]);
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V], ff[V];
        load_f<TI, V>(src + c, a);
        factor(c, ff);
        finish(c, a, ff);
    }
}

// x = y / rms(y) * w with y = alpha * x + r + bias (in place, fp32); plain = x rounded to T.  A thread keeps its part of y
// in registers (STEPS vectors); longer rows are recomputed in the second pass.
template <typename T, int V, int STEPS>
__global__ void scaled_norm_kernel(float* __restrict__ x, const T* __restrict__ r, int64_t r_stride, const float* __restrict__ bias,
                                   float alpha, const float* __restrict__ w, float eps, T* __restrict__ plain, int width) {
    const size_t t = blockIdx.x;
    float y[STEPS][V], ws[STEPS][V];
    float ss = 0.f;
    auto sum = [&](int c, float (&out)[V]) {
        float a[V];
        load_f<float, V>(x + t * width + c, out);
        load_f<T, V>(r + t * r_stride + c, a);
#pragma unroll
        for (int i = 0; i < V; i++) out[i] = fmaf(alpha, out[i], a[i]);
        if (bias) {
            load_f<float, V>(bias + c, a);
#pragma unroll
            for (int i = 0; i < V; i++) out[i] += a[i];
        }
    };
    const int stride = blockDim.x * V;
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) {
            load_f<float, V>(w + c, ws[s]);  // requested before the reduction
            sum(c, y[s]);
#pragma unroll
            for (int i = 0; i < V; i++) ss = fmaf(y[s][i], y[s][i], ss);
        }
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V];
        sum(c, a);
#pragma unroll
        for (int i = 0; i < V; i++) ss = fmaf(a[i], a[i], ss);
    }
    const float inv = 1.f / sqrtf(block_sum(ss) / width + eps);
    auto finish = [&](int c, float (&a)[V], const float (&ww)[V]) {
#pragma unroll
        for (int i = 0; i < V; i++) a[i] *= inv * ww[i];
        store_f<float, V>(x + t * width + c, a);
        if (plain) store_f<T, V>(plain + t * width + c, a);
    };
#pragma unroll
    for (int s = 0; s < STEPS; s++) {
        const int c = threadIdx.x * V + s * stride;
        if (c < width) finish(c, y[s], ws[s]);
    }
    for (int c = threadIdx.x * V + STEPS * stride; c < width; c += stride) {
        float a[V], ww[V];
        sum(c, a);
        load_f<float, V>(w + c, ww);
        finish(c, a, ww);
    }
}

// x[t] = table[ids[t]] * scale in fp32: the start of the residual stream; plain = x rounded to T
template <typename T, int V>
__global__ void embed_rows_kernel(float* __restrict__ x, T* __restrict__ plain, const T* __restrict__ table, const int32_t* __restrict__ ids,
                                  float scale, int width) {
    const T* src = table + (size_t)ids[blockIdx.x] * width;
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float a[V];
        load_f<T, V>(src + c, a);
#pragma unroll
        for (int i = 0; i < V; i++) a[i] *= scale;
        store_f<float, V>(x + (size_t)blockIdx.x * width + c, a);
        if (plain) store_f<T, V>(plain + (size_t)blockIdx.x * width + c, a);
    }
}

// out = g sigmoid(slope g) (u + 1), g = min(gate + bias, limit), u = clamp(up + bias, -limit, limit); a row of `in` is gate | up
template <typename T, int V>
__global__ void clamped_glu_kernel(T* __restrict__ out, const T* __restrict__ in, int64_t in_stride, const float* __restrict__ bias,
                                   float limit, float slope, int width) {
    const size_t t = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    if (c >= width) return;
    float g[V], u[V], bg[V], bu[V];
    load_f<T, V>(in + t * in_stride + c, g);
    load_f<T, V>(in + t * in_stride + width + c, u);
    load_f<float, V>(bias + c, bg);
    load_f<float, V>(bias + width + c, bu);
#pragma unroll
    for (int k = 0; k < V; k++) {
        const float a = fminf(g[k] + bg[k], limit), b = fminf(fmaxf(u[k] + bu[k], -limit), limit);
        g[k] = a * sigmoid_for<T>(slope * a) * (b + 1.f);
    }
    store_f<T, V>(out + t * width + c, g);
}

template <int V> __global__ void softcap_kernel(float* __restrict__ z, float cap, int64_t n) {
    const int64_t i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (i >= n) return;
    float a[V];
    load_f<float, V>(z + i, a);
#pragma unroll
    for (int k = 0; k < V; k++) a[k] = cap * tanhf(a[k] / cap);
    store_f<float, V>(z + i, a);
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
    // (1 + tanh u) / 2 = 1 / (1 + exp(-2u)); one exponential and one division
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return __fdividef(z, 1.f + exp2f(-2.885390081777927f * u));
}

template <typename T, int V>
__global__ void gelu_rows_kernel(T* __restrict__ out, const T* __restrict__ in, int64_t in_stride, int width) {
    const size_t t = blockIdx.x;
    for (int c = threadIdx.x * V; c < width; c += blockDim.x * V) {
        float a[V];
        load_f<T, V>(in + t * in_stride + c, a);
#pragma unroll
        for (int k = 0; k < V; k++) a[k] = gelu_tanh_f(a[k]);
        store_f<T, V>(out + t * width + c, a);
    }
}

int row_threads(int units) {
    int t = (units + 31) / 32 * 32;
    return t < 64 ? 64 : (t > 512 ? 512 : t);
}
bool aligned16(const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; }
int fail(const char* msg, int code = CA_ERR_INVALID) {
    set_last_error(msg);
    return code;
}
int done() {
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? CA_OK : fail(cudaGetErrorString(e), CA_ERR_CUDA);
}

bool aligned32(const void* p) { return reinterpret_cast<uintptr_t>(p) % 32 == 0; }

// calls f(T value, integral_constant V): V elements per access (wide: 8 of a 16-bit type)
template <typename F> int by_type(int dtype, bool vec, F&& f, bool wide = false) {
    if (dtype == CA_DTYPE_BF16) {
        if (vec && wide) f(__nv_bfloat16(), std::integral_constant<int, 8>());
        else if (vec) f(__nv_bfloat16(), std::integral_constant<int, 4>());
        else f(__nv_bfloat16(), std::integral_constant<int, 1>());
    } else if (dtype == CA_DTYPE_F16) {
        if (vec) f(__half(), std::integral_constant<int, 4>());
        else f(__half(), std::integral_constant<int, 1>());
    } else if (dtype == CA_DTYPE_F32) {
        if (vec) f(float(), std::integral_constant<int, 4>());
        else f(float(), std::integral_constant<int, 1>());
    } else {
        return fail("unknown element type");
    }
    return done();
}

}  // namespace
}  // namespace ca

using namespace ca;

extern "C" {

int ca_token_shift(const float* x, const float* mu, float* state, void* plain, void* shifted, const ca_spans* sp, int width,
                   int dtype, ca_stream stream) {
    if (!sp || width <= 0) return fail("token_shift: bad shape");
    if (sp->n_tokens == 0) return CA_OK;
    if (!x || !mu || !state || !plain || !shifted) return fail("token_shift: null pointer");
    const bool vec = width % 4 == 0 && aligned16(x) && aligned16(mu) && aligned16(state) && aligned16(plain) && aligned16(shifted);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        token_shift_kernel<T, V><<<sp->n_tokens, row_threads(width / V), 0, static_cast<cudaStream_t>(stream)>>>(
            x, mu, state, static_cast<T*>(plain), static_cast<T*>(shifted), *sp, width);
    });
}

int ca_gated_norm_add(float* x, const void* r, int64_t r_stride, const void* gate, int64_t gate_stride, const float* bias,
                      const float* weight, float eps, void* plain, const float* next_mu, float* next_state, void* next_shifted,
                      const ca_spans* sp, int64_t n_tokens, int width, int dtype, ca_stream stream) {
    if (n_tokens < 0 || width <= 0) return fail("gated_norm_add: bad shape");
    if (n_tokens == 0) return CA_OK;
    if (!x || !r || !gate || !bias || !weight) return fail("gated_norm_add: null pointer");
    if (next_mu && (!sp || !next_state || !next_shifted || sp->n_tokens != sp->n_entries || sp->n_tokens != n_tokens))
        return fail("gated_norm_add: the fused token shift needs one token per span");
    const bool vec = width % 4 == 0 && r_stride % 4 == 0 && gate_stride % 4 == 0 && aligned16(x) && aligned16(r) && aligned16(gate) &&
                     aligned16(bias) && aligned16(weight) && aligned16(plain) && aligned16(next_mu) && aligned16(next_state) &&
                     aligned16(next_shifted);
    const ca_spans spans = sp ? *sp : ca_spans{};
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        gated_norm_add_kernel<T, V, V == 1 ? 4 : (V == 8 ? 1 : 2)><<<(unsigned)n_tokens, row_threads(width / V), 0, static_cast<cudaStream_t>(stream)>>>(
            x, static_cast<const T*>(r), r_stride, static_cast<const T*>(gate), gate_stride, bias, weight, eps, static_cast<T*>(plain),
            next_mu, next_state, static_cast<T*>(next_shifted), spans, width);
    }, n_tokens <= 512 && width % 8 == 0 && r_stride % 8 == 0 && gate_stride % 8 == 0 && aligned32(x) && aligned32(bias) && aligned32(weight) &&
           aligned32(next_mu) && aligned32(next_state));
}

int ca_norm_rows(void* out, const void* x, int x_is_f32, int64_t x_stride, const int32_t* rows, const float* weight,
                 const void* gate, int64_t gate_stride, float eps, int64_t n_rows, int width, int dtype, ca_stream stream) {
    if (n_rows < 0 || width <= 0) return fail("norm_rows: bad shape");
    if (n_rows == 0) return CA_OK;
    if (!out || !x || !weight) return fail("norm_rows: null pointer");
    const bool vec = width % 4 == 0 && x_stride % 4 == 0 && (!gate || gate_stride % 4 == 0) && aligned16(out) && aligned16(x) &&
                     aligned16(weight) && aligned16(gate);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        const int threads = row_threads(width / V);
        if (x_is_f32)
            norm_rows_kernel<float, T, V><<<(unsigned)n_rows, threads, 0, static_cast<cudaStream_t>(stream)>>>(
                static_cast<T*>(out), static_cast<const float*>(x), x_stride, rows, weight, static_cast<const T*>(gate), gate_stride, eps, width);
        else
            norm_rows_kernel<T, T, V><<<(unsigned)n_rows, threads, 0, static_cast<cudaStream_t>(stream)>>>(
                static_cast<T*>(out), static_cast<const T*>(x), x_stride, rows, weight, static_cast<const T*>(gate), gate_stride, eps, width);
    }, width % 8 == 0 && x_stride % 8 == 0 && (!gate || gate_stride % 8 == 0) && aligned32(x) && aligned32(weight));
}

int ca_embed_rows(float* x, void* plain, const void* table, const int32_t* ids, float scale, int64_t n_tokens, int width, int dtype,
                  ca_stream stream) {
    if (n_tokens < 0 || width <= 0) return fail("embed_rows: bad shape");
    if (n_tokens == 0) return CA_OK;
    if (!x || !table || !ids) return fail("embed_rows: null pointer");
    const bool vec = width % 4 == 0 && aligned16(x) && aligned16(table) && aligned16(plain);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        embed_rows_kernel<T, V><<<(unsigned)n_tokens, row_threads(width / V), 0, static_cast<cudaStream_t>(stream)>>>(
            x, static_cast<T*>(plain), static_cast<const T*>(table), ids, scale, width);
    });
}

int ca_scaled_norm(float* x, const void* r, int64_t r_stride, const float* bias, float alpha, const float* weight, float eps, void* plain,
                   int64_t n_tokens, int width, int dtype, ca_stream stream) {
    if (n_tokens < 0 || width <= 0) return fail("scaled_norm: bad shape");
    if (n_tokens == 0) return CA_OK;
    if (!x || !r || !weight) return fail("scaled_norm: null pointer");
    const bool vec = width % 4 == 0 && r_stride % 4 == 0 && aligned16(x) && aligned16(r) && aligned16(bias) && aligned16(weight) && aligned16(plain);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        scaled_norm_kernel<T, V, V == 1 ? 4 : (V == 8 ? 1 : 2)><<<(unsigned)n_tokens, row_threads(width / V), 0, static_cast<cudaStream_t>(stream)>>>(
            x, static_cast<const T*>(r), r_stride, bias, alpha, weight, eps, static_cast<T*>(plain), width);
    }, width % 8 == 0 && r_stride % 8 == 0 && aligned32(x) && aligned32(bias) && aligned32(weight));
}

int ca_clamped_glu(void* out, const void* in, int64_t in_stride, const float* bias, float limit, float slope, int64_t n_rows, int width,
                   int dtype, ca_stream stream) {
    if (n_rows < 0 || width <= 0) return fail("clamped_glu: bad shape");
    if (n_rows == 0) return CA_OK;
    if (!out || !in || !bias) return fail("clamped_glu: null pointer");
    const bool vec = width % 4 == 0 && in_stride % 4 == 0 && aligned16(out) && aligned16(in) && aligned16(bias);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        const int units = (width + V - 1) / V, threads = units >= 256 ? 256 : row_threads(units);
        clamped_glu_kernel<T, V><<<dim3((unsigned)n_rows, (units + threads - 1) / threads), threads, 0, static_cast<cudaStream_t>(stream)>>>(
            static_cast<T*>(out), static_cast<const T*>(in), in_stride, bias, limit, slope, width);
    }, width % 8 == 0 && in_stride % 8 == 0 && aligned32(bias));
}

int ca_softcap(float* z, float cap, int64_t n, ca_stream stream) {
    if (n < 0 || !(cap > 0.f)) return fail("softcap: bad size or cap");
    if (n == 0) return CA_OK;
    if (!z) return fail("softcap: null pointer");
    const int V = n % 4 == 0 && aligned16(z) ? 4 : 1;
    const int64_t blocks = (n / V + 255) / 256;
    if (blocks > 0x7fffffff) return fail("softcap: too many elements");
    if (V == 4) softcap_kernel<4><<<(unsigned)blocks, 256, 0, static_cast<cudaStream_t>(stream)>>>(z, cap, n);
    else softcap_kernel<1><<<(unsigned)blocks, 256, 0, static_cast<cudaStream_t>(stream)>>>(z, cap, n);
    return done();
}

int ca_gelu_tanh(void* out, const void* in, int64_t in_stride, int64_t n_rows, int width, int dtype, ca_stream stream) {
    if (n_rows < 0 || width <= 0) return fail("gelu_tanh: bad shape");
    if (n_rows == 0) return CA_OK;
    if (!out || !in) return fail("gelu_tanh: null pointer");
    const bool vec = width % 4 == 0 && in_stride % 4 == 0 && aligned16(out) && aligned16(in);
    return by_type(dtype, vec, [&](auto tv, auto vv) {
        using T = decltype(tv);
        constexpr int V = decltype(vv)::value;
        gelu_rows_kernel<T, V><<<(unsigned)n_rows, row_threads(width / V), 0, static_cast<cudaStream_t>(stream)>>>(
            static_cast<T*>(out), static_cast<const T*>(in), in_stride, width);
    }, width % 8 == 0 && in_stride % 8 == 0);
}

}  // extern "C"
