// Causal grouped-query attention over the paged cache, one warp a (row, head).
//
// For the new row at position p of the sequence in `slot`, head h reads kv head
// g = h / (H / G) and sees cached positions lo..p, where lo is 0, or p + 1 - window (a
// sliding window), or the first position of p's chunk, floor(p / chunk) * chunk (chunks are
// counted from the sequence's position 0), whichever is later:
//   s_t = (q . k_t) * scale;  out = sum_t softmax(s)_t v_t
// Where a table of biases by distance is given (see common.cuh), the head's number for p - t is added to s_t.
// Keys have D values a head and values DV, which may differ.
// (crates/bc-infer/src/model.rs:448-481).  Like the reference's kernel
// (crates/bc-infer/src/gpu/kernels.h:271-324) it keeps a running maximum m, a running sum
// l and a running weighted sum of values, rescaled by e^(m - m') when a tile of positions
// raises the maximum; scores go lanes-over-positions, values lanes-over-dimensions.  The
// order of every sum depends only on the position index, so a row's result is the same
// bits whether it came in a prompt, alone, or beside other sequences.  This kernel serves
// the true 32-bit path for prompts and decoding alike, and stands as the checked twin of
// the faster bf16 kernels.
//
// Cache layout of one layer: keys [page][kv_head][BC_PAGE][D], values [page][kv_head][BC_PAGE][DV]; page_table[slot][i] names the
// page of positions 64 i .. 64 i + 63.  Rows whose slot is negative are padding: their
// output is zero.
#include "common.cuh"

#define WARPS 4
#define MAX_D 256

template <class T> struct KeyDot;
template <> struct KeyDot<float> {
    static __device__ __forceinline__ float dot(const float* k, const float* q, int D) {
        float s = 0.0f;
        for (int d = 0; d < D; d += 4) {
            const float4 kv = *reinterpret_cast<const float4*>(k + d);
            const float4 qv = *reinterpret_cast<const float4*>(q + d);
            s = fmaf(kv.x, qv.x, s); s = fmaf(kv.y, qv.y, s); s = fmaf(kv.z, qv.z, s); s = fmaf(kv.w, qv.w, s);
        }
        return s;
    }
};
template <> struct KeyDot<bf16> {
    static __device__ __forceinline__ float dot(const bf16* k, const float* q, int D) {
        float s = 0.0f;
        for (int d = 0; d < D; d += 8) {
            const uint4 kv = *reinterpret_cast<const uint4*>(k + d);
            const float4 q0 = *reinterpret_cast<const float4*>(q + d);
            const float4 q1 = *reinterpret_cast<const float4*>(q + d + 4);
            s = fmaf(__uint_as_float(kv.x << 16), q0.x, s); s = fmaf(__uint_as_float(kv.x & 0xffff0000u), q0.y, s);
            s = fmaf(__uint_as_float(kv.y << 16), q0.z, s); s = fmaf(__uint_as_float(kv.y & 0xffff0000u), q0.w, s);
            s = fmaf(__uint_as_float(kv.z << 16), q1.x, s); s = fmaf(__uint_as_float(kv.z & 0xffff0000u), q1.y, s);
            s = fmaf(__uint_as_float(kv.w << 16), q1.z, s); s = fmaf(__uint_as_float(kv.w & 0xffff0000u), q1.w, s);
        }
        return s;
    }
};

// Head sizes that are no multiple of 8: element by element, in the same ascending order.
template <class T> __device__ __forceinline__ float dot_any(const T* k, const float* q, int D) {
    float s = 0.0f;
    for (int d = 0; d < D; d++) s = fmaf(to_f32(k[d]), q[d], s);
    return s;
}

template <class T>
__global__ void __launch_bounds__(WARPS * 32) attention_rows_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k_cache,
                                                                   const T* __restrict__ v_cache, const int* __restrict__ page_table,
                                                                   const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                                                                   T* __restrict__ out, int H, int G, int D, int DV, int max_pages,
                                                                   int n_pages, int window, int chunk, float scale, int sink, float out_scale,
                                                                   const float* __restrict__ bias, int bias_reach) {
    __shared__ __align__(16) float qs[WARPS][MAX_D];
    pdl_launch_dependents();
    pdl_wait();
    PDL_FRESH(q); PDL_FRESH(k_cache); PDL_FRESH(v_cache);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = blockIdx.x, h = blockIdx.y * WARPS + warp;
    if (h >= H) return;
    T* o = out + ((size_t)r * H + h) * DV;
    const int slot = row_slot[r];
    const int nd = (DV + 31) / 32;
    if (slot < 0) {
        for (int j = 0; j < nd; j++)
            if (lane + 32 * j < DV) o[lane + 32 * j] = from_f32<T>(0.0f);
        return;
    }
    const int pos = row_pos[r];
    const int g = h / (H / G);
    const float* hb = bias == nullptr ? nullptr : bias_of_kv_head(bias, bias_reach, H / G, g) + h % (H / G);
    const T* qh = q + (size_t)r * q_stride + (size_t)h * D;
    for (int d = lane; d < D; d += 32) qs[warp][d] = to_f32(qh[d]);
    __syncwarp();

    int lo = window > 0 && pos + 1 > window ? pos + 1 - window : 0;
    if (chunk > 0) lo = max(lo, pos / chunk * chunk);
    const int* pages = page_table + (size_t)slot * max_pages;
    float acc[MAX_D / 32];
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) acc[j] = 0.0f;
    float m = -INFINITY, l = 0.0f;
    for (int t0 = lo & ~31; t0 <= pos; t0 += 32) {
        // A tile of 32 positions starts at a multiple of 32, so it lies in one page.
        const int pi = t0 / BC_PAGE;
        int page = pi < max_pages ? pages[pi] : -1;
        if (page < 0 || page >= n_pages) page = -1;
        const size_t at = ((size_t)(page < 0 ? 0 : page) * G + g) * BC_PAGE + (t0 % BC_PAGE);
        const size_t base = at * D;
        const int t = t0 + lane;
        const bool seen = page >= 0 && t >= lo && t <= pos;
        float s = -INFINITY;
        if (seen) s = (D % 8 == 0 ? KeyDot<T>::dot(k_cache + base + (size_t)lane * D, qs[warp], D) : dot_any<T>(k_cache + base + (size_t)lane * D, qs[warp], D)) * scale;
        if (seen && hb != nullptr) s += hb[(size_t)min(pos - t, bias_reach - 1) * (H / G)];
        const float mn = fmaxf(m, warp_max(s));
        const float corr = mn == -INFINITY ? 1.0f : expf(m - mn);
        const float p = seen ? expf(s - mn) : 0.0f;
        l = l * corr + warp_sum(p);
#pragma unroll
        for (int j = 0; j < MAX_D / 32; j++) acc[j] *= corr;
        const int count = page < 0 ? 0 : min(32, pos + 1 - t0);
        const T* vt = v_cache + at * DV;
        for (int i = max(0, lo - t0); i < count; i++) {
            const float pi_ = __shfl_sync(0xffffffffu, p, i);
#pragma unroll
            for (int j = 0; j < MAX_D / 32; j++) {
                const int d = lane + 32 * j;
                if (j < nd && d < DV) acc[j] = fmaf(pi_, to_f32(vt[(size_t)i * DV + d]), acc[j]);
            }
        }
        m = mn;
    }
    // A sink is one more position of score 0 that has no value: it adds e^(0 - m) to the sum of the weights alone.
    if (sink && m != -INFINITY) l += expf(-m);
    const float inv = l > 0.0f ? out_scale / l : 0.0f;
#pragma unroll
    for (int j = 0; j < MAX_D / 32; j++) {
        const int d = lane + 32 * j;
        if (j < nd && d < DV) o[d] = from_f32<T>(acc[j] * inv);
    }
}

template <class T>
static int launch(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table, const int* row_pos,
                  const int* row_slot, void* out, int rows, int H, int G, int D, int DV, int max_pages, int n_pages, int window, int chunk,
                  float scale, int sink, float out_scale, const float* bias, int bias_reach, cudaStream_t s) {
    BC_CHECK_ARG(bias == nullptr || bias_reach > 0, "attention_rows: a table of biases for %d distances", bias_reach);
    BC_CHECK_ARG(rows >= 0 && H > 0 && G > 0 && H % G == 0, "attention_rows: bad sizes rows=%d H=%d G=%d", rows, H, G);
    BC_CHECK_ARG(D > 0 && D <= MAX_D, "attention_rows: head size %d is not within 1 to %d", D, MAX_D);
    BC_CHECK_ARG(DV > 0 && DV <= MAX_D && window >= 0 && chunk >= 0, "attention_rows: bad value width %d, window %d or chunk %d", DV, window, chunk);
    BC_CHECK_ARG(rows <= 2147483647 && (H + WARPS - 1) / WARPS <= 65535, "attention_rows: too many heads (%d)", H);
    if (rows == 0) return BC_OK;
    dim3 grid(rows, (H + WARPS - 1) / WARPS);
    bc_launch(attention_rows_kernel<T>, grid, dim3(WARPS * 32), 0, s, (const T*)q, q_stride, (const T*)k_cache, (const T*)v_cache, page_table,
              row_pos, row_slot, (T*)out, H, G, D, DV, max_pages, n_pages, window, chunk, scale, sink, out_scale, bias, bias_reach);
    BC_LAUNCH_STATUS();
}

// q: row r's head h at q + r * q_stride + h * D (so q may live inside a fused projection).
extern "C" int bc_attention_rows_f32(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                     const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int max_pages,
                                     int n_pages, int window, float scale, cudaStream_t s) {
    return launch<float>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, D, max_pages, n_pages, window, 0, scale, 0, 1.0f, nullptr, 0, s);
}
extern "C" int bc_attention_rows_bf16(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                      const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int max_pages,
                                      int n_pages, int window, float scale, cudaStream_t s) {
    return launch<bf16>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, D, max_pages, n_pages, window, 0, scale, 0, 1.0f, nullptr, 0, s);
}

// The same with values of their own width DV (out: [rows, H, DV]) and a chunk mask beside the window (0: none).
extern "C" int bc_attention_rows_kv_f32(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                        const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int DV, int max_pages,
                                        int n_pages, int window, int chunk, float scale, cudaStream_t s) {
    return launch<float>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, chunk, scale, 0, 1.0f, nullptr, 0, s);
}
extern "C" int bc_attention_rows_kv_bf16(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                         const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int DV, int max_pages,
                                         int n_pages, int window, int chunk, float scale, cudaStream_t s) {
    return launch<bf16>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, chunk, scale, 0, 1.0f, nullptr, 0, s);
}

// The same with a sink (one more position of score 0 without a value, so that the weights of a row add up to less
// than one), a factor on the output, and biases by distance: a table as in common.cuh
// (null: none).
extern "C" int bc_attention_rows_sink_f32(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                          const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int DV, int max_pages,
                                          int n_pages, int window, int chunk, float scale, int sink, float out_scale, const float* bias, int bias_reach,
                                          cudaStream_t s) {
    return launch<float>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, chunk, scale, sink, out_scale, bias, bias_reach, s);
}
extern "C" int bc_attention_rows_sink_bf16(const void* q, int q_stride, const void* k_cache, const void* v_cache, const int* page_table,
                                           const int* row_pos, const int* row_slot, void* out, int rows, int H, int G, int D, int DV, int max_pages,
                                           int n_pages, int window, int chunk, float scale, int sink, float out_scale, const float* bias, int bias_reach,
                                          cudaStream_t s) {
    return launch<bf16>(q, q_stride, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, chunk, scale, sink, out_scale, bias, bias_reach, s);
}
