// What enters the residual stream where a row is a sum: the token's embedding, a second embedding named by the token and the one
// before it, and a sinusoidal vector of the position.  Each of the three may be left out; without the token's table the others are
// added to what the stream already holds.
//
//   x[r] = table[t] * scale + pairs[b] + s(p)
//   b = (before * mul_prev + t * mul_cur) mod buckets;  at a sequence's first position b = buckets, the table's last row
//   s(p)[2 i] = sin(p f_i), s(p)[2 i + 1] = cos(p f_i)
//
// The token before is the row ahead in the same step, or, for the first row a sequence brings, what an earlier step left in the
// sequence's pages: every row writes its own token there (one int32 a position, [page][64]).  A row reads position p - 1 and writes
// position p, so no row reads what another row of the same step writes.
//
// Angles: p f_i in double, taken back into one turn there; sine and cosine of that in float.
#include "common.cuh"

template <class T> struct PairLoad;
template <> struct PairLoad<float> {
    static __device__ __forceinline__ float2 at(const float* p) { return *reinterpret_cast<const float2*>(p); }
};
template <> struct PairLoad<bf16> {
    static __device__ __forceinline__ float2 at(const bf16* p) {
        const uint32_t raw = *reinterpret_cast<const uint32_t*>(p);
        return make_float2(__uint_as_float(raw << 16), __uint_as_float(raw & 0xffff0000u));
    }
};

__device__ __forceinline__ float2 turn(int pos, double f) {
    double a = (double)pos * f;
    a -= rint(a * 0.15915494309189535) * 6.283185307179586;
    float s, c;
    sincosf((float)a, &s, &c);
    return make_float2(s, c);
}

template <class T>
__global__ void __launch_bounds__(256)
embed_sum_kernel(const T* __restrict__ table, const int* __restrict__ tokens, int V, float scale, const T* __restrict__ pairs, int buckets,
                 long long mul_prev, long long mul_cur, const int* __restrict__ row_pos, const int* __restrict__ row_slot,
                 const int* __restrict__ page_table, int max_pages, int n_pages, int* history, const double* __restrict__ freq,
                 float* __restrict__ out, int E) {
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(tokens); PDL_FRESH(row_pos); PDL_FRESH(row_slot); PDL_FRESH(page_table); PDL_FRESH(out);
    const int r = blockIdx.x;
    const int t = tokens[r], pos = row_pos[r], slot = row_slot[r];
    const bool ok = t >= 0 && t < V;
    const T* src = table == nullptr ? nullptr : table + (size_t)(ok ? t : 0) * E;
    const T* pair = nullptr;
    if (pairs != nullptr && slot >= 0 && pos >= 0) {
        const int* pages = page_table + (size_t)slot * max_pages;
        long long before = -1;
        if (pos > 0) {
            if (r > 0 && row_slot[r - 1] == slot) {
                before = tokens[r - 1];
            } else if ((pos - 1) / BC_PAGE < max_pages) {
                const int page = pages[(pos - 1) / BC_PAGE];
                if (page >= 0 && page < n_pages) before = history[(size_t)page * BC_PAGE + (pos - 1) % BC_PAGE];
            }
        }
        const long long row = before < 0 ? buckets : (before * mul_prev + (long long)t * mul_cur) % buckets;
        pair = pairs + (size_t)row * E;
        if (threadIdx.x == 0 && pos / BC_PAGE < max_pages) {
            const int page = pages[pos / BC_PAGE];
            if (page >= 0 && page < n_pages) history[(size_t)page * BC_PAGE + pos % BC_PAGE] = t;
        }
    }
    float* dst = out + (size_t)r * E;
    if (E % 2 == 0) {
        for (int c = 2 * threadIdx.x; c < E; c += 2 * blockDim.x) {
            float2 v;
            if (src == nullptr) {
                v = *reinterpret_cast<const float2*>(dst + c);
            } else {
                v = ok ? PairLoad<T>::at(src + c) : make_float2(0.0f, 0.0f);
                v = make_float2(v.x * scale, v.y * scale);
            }
            if (pair != nullptr) {
                const float2 b = PairLoad<T>::at(pair + c);
                v = make_float2(v.x + b.x, v.y + b.y);
            }
            if (freq != nullptr) {
                const float2 a = turn(pos, freq[c / 2]);
                v = make_float2(v.x + a.x, v.y + a.y);
            }
            *reinterpret_cast<float2*>(dst + c) = v;
        }
        return;
    }
    for (int c = threadIdx.x; c < E; c += blockDim.x) {
        float v = src == nullptr ? dst[c] : ok ? to_f32(src[c]) * scale : 0.0f;
        if (pair != nullptr) v += to_f32(pair[c]);
        if (freq != nullptr) {
            const float2 a = turn(pos, freq[c / 2]);
            v += c % 2 ? a.y : a.x;
        }
        dst[c] = v;
    }
}

// table: [V, E] or null (out is then added to); pairs: [buckets + 1, E] or null; history: [pages, 64] int32, with page_table
// [slots, max_pages] (both used with pairs only); freq: [(E + 1) / 2] double or null; out: [rows, E] float.
template <class T>
static int embed_sum(const void* table, const int* tokens, int V, float scale, const void* pairs, int buckets, long long mul_prev, long long mul_cur,
                     const int* row_pos, const int* row_slot, const int* page_table, int max_pages, int n_pages, int* history, const double* freq,
                     float* out, int rows, int E, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && E > 0 && V > 0, "embed_sum: bad sizes rows=%d E=%d V=%d", rows, E, V);
    BC_CHECK_ARG(pairs == nullptr || (buckets > 0 && history && page_table && max_pages > 0 && n_pages > 0), "embed_sum: pairs of tokens need %d > 0 rows, pages and a table of them", buckets);
    BC_CHECK_ARG(mul_prev >= 0 && mul_cur >= 0 && mul_prev < (1ll << 31) && mul_cur < (1ll << 31), "embed_sum: the factors must lie in 0 .. 2^31 - 1");
    if (rows == 0) return BC_OK;
    const int n = E % 2 ? E : E / 2;
    bc_launch(embed_sum_kernel<T>, dim3(rows), dim3(n <= 64 ? 64 : n <= 128 ? 128 : 256), 0, s, (const T*)table, tokens, V, scale, (const T*)pairs, buckets,
              mul_prev, mul_cur, row_pos, row_slot, page_table, max_pages, n_pages, history, freq, out, E);
    BC_LAUNCH_STATUS();
}
extern "C" int bc_embed_sum_f32(const void* table, const int* tokens, int V, float scale, const void* pairs, int buckets, long long mul_prev,
                                long long mul_cur, const int* row_pos, const int* row_slot, const int* page_table, int max_pages, int n_pages,
                                int* history, const double* freq, float* out, int rows, int E, cudaStream_t s) {
    return embed_sum<float>(table, tokens, V, scale, pairs, buckets, mul_prev, mul_cur, row_pos, row_slot, page_table, max_pages, n_pages, history, freq, out,
                            rows, E, s);
}
extern "C" int bc_embed_sum_bf16(const void* table, const int* tokens, int V, float scale, const void* pairs, int buckets, long long mul_prev,
                                 long long mul_cur, const int* row_pos, const int* row_slot, const int* page_table, int max_pages, int n_pages,
                                 int* history, const double* freq, float* out, int rows, int E, cudaStream_t s) {
    return embed_sum<bf16>(table, tokens, V, scale, pairs, buckets, mul_prev, mul_cur, row_pos, row_slot, page_table, max_pages, n_pages, history, freq, out,
                           rows, E, s);
}
