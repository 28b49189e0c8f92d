// A residual stream of several copies a row (hyper-connections): between two sublayers of a model whose rows carry a bundle
// X [S, E] of float streams, with a connection (in [S], mix [S, S] indexed [from, to], out [S]) around every sublayer,
//
//   X_t <- sum_s mix[s][t] X_s + out[t] * scale * y        the sublayer before leaves its result y (scale [E], or none)
//   u = sum_t in[t] X_t                                     the next sublayer enters
//   h = u / sqrt(mean(u^2) + eps) * w                       its norm, in the activation type
//
// is ONE kernel, a block a row: the streams are read and written once, y is cleared for the next sublayer's product to add into.
// Nothing pending (the first sublayer): only the second and third line.  No `in`: every stream counts once (the model's end),
// and with a list of rows only those are read and nothing but h is written.
//
//   start     X_s = e / sqrt(mean(e^2) + eps) * w for every s, from the embedded rows e
//
// Everything is float up to h.  A row's sums run in an order that its width alone fixes.
#include "common.cuh"

#define HS_MAX_STREAMS 64

__device__ __forceinline__ float4 hs_fma(float a, float4 b, float4 c) {
    return make_float4(fmaf(a, b.x, c.x), fmaf(a, b.y, c.y), fmaf(a, b.z, c.z), fmaf(a, b.w, c.w));
}
__device__ __forceinline__ float hs_fma(float a, float b, float c) { return fmaf(a, b, c); }
__device__ __forceinline__ float hs_square(float4 v) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w))); }
__device__ __forceinline__ float hs_square(float v) { return v * v; }
__device__ __forceinline__ float4 hs_mul(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }
__device__ __forceinline__ float hs_mul(float a, float b) { return a * b; }
template <class V> __device__ __forceinline__ V hs_zero();
template <> __device__ __forceinline__ float hs_zero<float>() { return 0.0f; }
template <> __device__ __forceinline__ float4 hs_zero<float4>() { return make_float4(0.0f, 0.0f, 0.0f, 0.0f); }

__device__ __forceinline__ void hs_store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void hs_store(bf16* p, float4 v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
}
template <class T> __device__ __forceinline__ void hs_store(T* p, float v) { *p = from_f32<T>(v); }

// V: float4 where the width is a multiple of 4, else float.  SS > 0: the number of streams; 0: any number up to HS_MAX_STREAMS.
template <int SS, class V, class T>
__global__ void __launch_bounds__(512)
hyper_step_kernel(float* x, float* y, const float* __restrict__ scale, const float* __restrict__ mix, const float* __restrict__ out_w,
                  const float* __restrict__ in_w, const float* __restrict__ w, const int* __restrict__ gather, T* __restrict__ h, int S_any, int E,
                  int x_rows, float eps) {
    constexpr int N = SS > 0 ? SS : HS_MAX_STREAMS;
    constexpr int W = sizeof(V) / 4;
    const int S = SS > 0 ? SS : S_any;
    extern __shared__ __align__(16) float u_row[];          // the collapsed row, [E]
    __shared__ float scratch[32];
    __shared__ float m_s[N * N], o_s[N], i_s[N];
    const bool pending = y != nullptr;
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) m_s[i] = pending ? mix[i] : 0.0f;
    for (int i = threadIdx.x; i < S; i += blockDim.x) {
        o_s[i] = pending ? out_w[i] : 0.0f;
        i_s[i] = in_w ? in_w[i] : 1.0f;
    }
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(x); PDL_FRESH(y);
    __syncthreads();
    const int row = gather ? gather[blockIdx.x] : blockIdx.x;
    if (row < 0 || row >= x_rows) return;
    float* xr = x + (size_t)row * S * E;
    float* yr = pending ? y + (size_t)row * E : nullptr;
    float ss = 0.0f;
#pragma unroll 2
    for (int c = W * threadIdx.x; c < E; c += W * blockDim.x) {
        V in[N];
        if (SS > 0) {
#pragma unroll
            for (int s = 0; s < N; s++) in[s] = *reinterpret_cast<const V*>(xr + (size_t)s * E + c);
        } else {
            for (int s = 0; s < S; s++) in[s] = *reinterpret_cast<const V*>(xr + (size_t)s * E + c);
        }
        V u = hs_zero<V>();
        if (pending) {
            V v = *reinterpret_cast<const V*>(yr + c);
            if (scale) v = hs_mul(v, *reinterpret_cast<const V*>(scale + c));
            if (!gather) *reinterpret_cast<V*>(yr + c) = hs_zero<V>();
            auto one = [&](int t) {
                V a = hs_zero<V>();
                if (SS > 0) {
#pragma unroll
                    for (int s = 0; s < N; s++) a = hs_fma(m_s[s * S + t], in[s], a);
                } else {
                    for (int s = 0; s < S; s++) a = hs_fma(m_s[s * S + t], in[s], a);
                }
                a = hs_fma(o_s[t], v, a);
                if (!gather) *reinterpret_cast<V*>(xr + (size_t)t * E + c) = a;
                u = hs_fma(i_s[t], a, u);
            };
            if (SS > 0) {
#pragma unroll
                for (int t = 0; t < N; t++) one(t);
            } else {
                for (int t = 0; t < S; t++) one(t);
            }
        } else {
            if (SS > 0) {
#pragma unroll
                for (int t = 0; t < N; t++) u = hs_fma(i_s[t], in[t], u);
            } else {
                for (int t = 0; t < S; t++) u = hs_fma(i_s[t], in[t], u);
            }
        }
        *reinterpret_cast<V*>(u_row + c) = u;             // read back by the same thread alone
        ss += hs_square(u);
    }
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)E + eps);
    T* hr = h + (size_t)blockIdx.x * E;
    for (int c = W * threadIdx.x; c < E; c += W * blockDim.x) {
        const V g = hs_mul(*reinterpret_cast<const V*>(u_row + c), *reinterpret_cast<const V*>(w + c));
        hs_store(hr + c, hs_fma(f, g, hs_zero<V>()));
    }
}

template <class V>
__global__ void __launch_bounds__(512)
hyper_start_kernel(const float* e, const float* __restrict__ w, float* __restrict__ x, int S, int E, float eps) {
    constexpr int W = sizeof(V) / 4;
    __shared__ float scratch[32];
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(e);
    const float* er = e + (size_t)blockIdx.x * E;
    float* xr = x + (size_t)blockIdx.x * S * E;
    float ss = 0.0f;
    for (int c = W * threadIdx.x; c < E; c += W * blockDim.x) ss += hs_square(*reinterpret_cast<const V*>(er + c));
    const float f = w ? 1.0f / sqrtf(block_sum(ss, scratch) / (float)E + eps) : 1.0f;
    for (int c = W * threadIdx.x; c < E; c += W * blockDim.x) {
        V v = *reinterpret_cast<const V*>(er + c);
        if (w) v = hs_fma(f, hs_mul(v, *reinterpret_cast<const V*>(w + c)), hs_zero<V>());
        for (int s = 0; s < S; s++) *reinterpret_cast<V*>(xr + (size_t)s * E + c) = v;
    }
}

// By the width alone: about two vectors a thread.
static int hs_threads(int E) {
    const int want = E % 4 == 0 ? E / 8 : E / 2;
    int t = 32;
    while (t < want && t < 512) t *= 2;
    return t;
}

template <class T>
static int hyper_step(float* x, float* y, const float* scale, const float* mix, const float* out_w, const float* in_w, const float* w, const int* gather,
                      void* h, int rows, int x_rows, int S, int E, float eps, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && x_rows >= 0 && E > 0 && E <= 32768 && eps > 0.0f, "hyper_step: bad sizes rows=%d E=%d eps=%g", rows, E, (double)eps);
    BC_CHECK_ARG(S >= 1 && S <= HS_MAX_STREAMS, "hyper_step: %d streams are outside 1 to %d", S, HS_MAX_STREAMS);
    BC_CHECK_ARG(!y || (mix && out_w), "hyper_step: a pending result comes with its connection");
    if (rows == 0) return BC_OK;        // nothing asked for (the list of rows is empty, and its pointer null)
    BC_CHECK_ARG(gather || rows == x_rows, "hyper_step: %d rows of %d without a list", rows, x_rows);
    const bool vec = E % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)y % 16 == 0 && (uintptr_t)scale % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)h % 16 == 0;
    const size_t smem = (size_t)E * sizeof(float);
    cudaError_t e = cudaSuccess;
#define HS_GO(SS, V)                                                                                                                          \
    do {                                                                                                                                      \
        static bool configured = false;                                                                                                       \
        if (!configured) {                                                                                                                    \
            e = cudaFuncSetAttribute(hyper_step_kernel<SS, V, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 32768 * 4);                    \
            configured = e == cudaSuccess;                                                                                                    \
        }                                                                                                                                     \
        if (e == cudaSuccess)                                                                                                                 \
            e = bc_launch(hyper_step_kernel<SS, V, T>, dim3(rows), dim3(hs_threads(E)), smem, s, x, y, scale, mix, out_w, in_w, w, gather, (T*)h, S, \
                          E, x_rows, eps);                                                                                                    \
    } while (0)
#define HS_CASE(SS)                       \
    case SS:                              \
        if (vec) HS_GO(SS, float4);       \
        else HS_GO(SS, float);            \
        break;
    switch (S) {
        HS_CASE(1) HS_CASE(2) HS_CASE(3) HS_CASE(4) HS_CASE(5) HS_CASE(6) HS_CASE(7) HS_CASE(8)
        default: HS_GO(0, float);
    }
#undef HS_CASE
#undef HS_GO
    if (e != cudaSuccess) {
        bc_set_error("hyper_step: %s", cudaGetErrorString(e));
        return (int)e;
    }
    BC_LAUNCH_STATUS();
}

// x: [x_rows, S, E] float; y (null: nothing pending): [x_rows, E] float; scale: [E] or null; mix: [S, S] (from, to); out_w, in_w: [S]
// (in_w null: ones); w: [E]; gather: rows to take, or null (all; then x is changed in place and y left as zeros); h: [rows, E].
extern "C" int bc_hyper_step_f32(float* x, float* y, const float* scale, const float* mix, const float* out_w, const float* in_w, const float* w,
                                 const int* gather, void* h, int rows, int x_rows, int S, int E, float eps, cudaStream_t s) {
    return hyper_step<float>(x, y, scale, mix, out_w, in_w, w, gather, h, rows, x_rows, S, E, eps, s);
}
extern "C" int bc_hyper_step_bf16(float* x, float* y, const float* scale, const float* mix, const float* out_w, const float* in_w, const float* w,
                                  const int* gather, void* h, int rows, int x_rows, int S, int E, float eps, cudaStream_t s) {
    return hyper_step<bf16>(x, y, scale, mix, out_w, in_w, w, gather, h, rows, x_rows, S, E, eps, s);
}

// e: [rows, E] float; w: [E] or null (no norm); x: [rows, S, E] float.
extern "C" int bc_hyper_start(const float* e, const float* w, float* x, int rows, int S, int E, float eps, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && E > 0 && S >= 1 && S <= HS_MAX_STREAMS, "hyper_start: bad sizes rows=%d S=%d E=%d", rows, S, E);
    if (rows == 0) return BC_OK;
    if (E % 4 == 0 && (uintptr_t)e % 16 == 0 && (uintptr_t)w % 16 == 0 && (uintptr_t)x % 16 == 0)
        bc_launch(hyper_start_kernel<float4>, dim3(rows), dim3(hs_threads(E)), 0, s, e, w, x, S, E, eps);
    else
        bc_launch(hyper_start_kernel<float>, dim3(rows), dim3(hs_threads(E)), 0, s, e, w, x, S, E, eps);
    BC_LAUNCH_STATUS();
}
