// Differential attention over the paged cache: every head holds two query maps, every kv head two key maps over one set of values,
//
//   A_m = sum_j softmax_j(scale q_{h,m} . k_{g,m}(j)) v_g(j),  m = 0, 1;     z = A_0 - lambda A_1;
//   out_h = z / sqrt(mean(z^2) + eps) * factor                               (no weight; the mean over the head's values)
//
// causal, grouped-query, with a window that keeps a sequence's first positions: a row at position i sees j <= i with i - j < window
// or j < keep (window 0: every j <= i).  Keys have D values a map, values DV.
//
//   rows    one warp a (row, head), both maps at once: the true 32-bit path for prompts and decoding alike, any size up to 256, and
//           the checked twin of the tile kernel
//   tiles   bf16 on m16n8k16 tensor-core tiles: a block takes (kv head, tile of rows, sequence); half of its warps multiply map 0 and
//           half map 1 of the same rows (tokens x the heads that share the kv head, token-major), so that a page of both key maps and
//           of values is fetched once for both.  The maps meet in shared memory at the end, where the difference, its norm and the
//           factor are taken in float before anything is rounded.  Steps of few rows a sequence share a row's pages out over several
//           blocks (`splits`), whose maxima, sums and products a second kernel merges in the order of the splits
//
// Cache of one layer: keys [page][2 kv_heads][BC_PAGE][D] (the maps of a kv head side by side), values [page][kv_heads][BC_PAGE][DV];
// page_table[slot][i] names the page of positions 64 i .. 64 i + 63.  Scores, weights and all sums are float; the tile kernel rounds
// the weights to bf16 for their product with the values.  A row's sums run in an order that its position and the sizes alone fix.
#include "common.cuh"
#include "mma_tiles.cuh"

#define DA_MAX_D 256
#define DA_WARPS 4          // rows kernel: heads a block

// The pages a stretch of rows reads, in order: those of the kept first positions, then those from `first` (the page of the oldest
// position the window of the stretch's first row shows) on.
struct DaPages {
    int kept, first, count;       // pages ahead of `first` that are read; first page of the window; pages in all
    __device__ __forceinline__ DaPages(int first_row_pos, int last_row_pos, int window, int keep) {
        const int end = last_row_pos / BC_PAGE + 1;
        const int lo = window > 0 && first_row_pos + 1 > window ? first_row_pos + 1 - window : 0;
        first = lo / BC_PAGE;
        kept = min(first, (keep + BC_PAGE - 1) / BC_PAGE);
        count = kept + (end - first);
    }
    __device__ __forceinline__ int page(int i) const { return i < kept ? i : first + (i - kept); }
};

// ---------------------------------------------------------------------------------------- rows
template <class T> __device__ __forceinline__ float da_dot(const T* k, const float* q, int D);
template <> __device__ __forceinline__ float da_dot<float>(const float* k, const float* q, int D) {
    float s = 0.0f;
    if (D % 4 == 0) {
        for (int d = 0; d < D; d += 4) {
            const float4 kv = *reinterpret_cast<const float4*>(k + d), qv = *reinterpret_cast<const float4*>(q + d);
            s = fmaf(kv.x, qv.x, s); s = fmaf(kv.y, qv.y, s); s = fmaf(kv.z, qv.z, s); s = fmaf(kv.w, qv.w, s);
        }
        return s;
    }
    for (int d = 0; d < D; d++) s = fmaf(k[d], q[d], s);
    return s;
}
template <> __device__ __forceinline__ float da_dot<bf16>(const bf16* k, const float* q, int D) {
    float s = 0.0f;
    if (D % 4 == 0) {
        for (int d = 0; d < D; d += 4) {
            const uint2 kv = *reinterpret_cast<const uint2*>(k + d);
            const float4 qv = *reinterpret_cast<const float4*>(q + d);
            s = fmaf(__uint_as_float(kv.x << 16), qv.x, s); s = fmaf(__uint_as_float(kv.x & 0xffff0000u), qv.y, s);
            s = fmaf(__uint_as_float(kv.y << 16), qv.z, s); s = fmaf(__uint_as_float(kv.y & 0xffff0000u), qv.w, s);
        }
        return s;
    }
    for (int d = 0; d < D; d++) s = fmaf(to_f32(k[d]), q[d], s);
    return s;
}

template <class T>
__global__ void __launch_bounds__(DA_WARPS * 32)
diff_rows_kernel(const T* q, const T* k_cache, const T* v_cache, const int* __restrict__ page_table, const int* __restrict__ row_pos,
                 const int* __restrict__ row_slot, T* __restrict__ out, int H, int G, int D, int DV, int max_pages, int n_pages, int window, int keep,
                 float scale, float lambda, float eps, float factor) {
    __shared__ __align__(16) float qs[DA_WARPS][2][DA_MAX_D];
    pdl_launch_dependents();
    pdl_wait();
    PDL_FRESH(q); PDL_FRESH(k_cache); PDL_FRESH(v_cache);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int r = blockIdx.x, h = blockIdx.y * DA_WARPS + warp;
    if (h >= H) return;
    T* o = out + ((size_t)r * H + h) * DV;
    const int slot = row_slot[r];
    if (slot < 0) {
        for (int d = lane; d < DV; d += 32) o[d] = from_f32<T>(0.0f);
        return;
    }
    const int pos = row_pos[r], g = h / (H / G);
    const T* qh = q + ((size_t)r * H + h) * 2 * D;
    for (int d = lane; d < 2 * D; d += 32) qs[warp][d / D][d % D] = to_f32(qh[d]);
    __syncwarp();
    const int lo = window > 0 && pos + 1 > window ? pos + 1 - window : 0;
    const int* pages = page_table + (size_t)slot * max_pages;
    float acc[2][DA_MAX_D / 32], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int j = 0; j < DA_MAX_D / 32; j++) acc[0][j] = acc[1][j] = 0.0f;
    const DaPages walk(pos, pos, window, keep);
    for (int it = 0; it < 2 * walk.count; it++) {
        const int t0 = walk.page(it >> 1) * BC_PAGE + (it & 1) * 32;       // a tile of 32 positions, half a page
        if (t0 > pos || (t0 + 31 < lo && t0 >= keep)) continue;
        const int pi = t0 / BC_PAGE;
        const int page = pi < max_pages ? pages[pi] : -1;
        if (page < 0 || page >= n_pages) continue;
        const int t = t0 + lane;
        const bool seen = t <= pos && (t >= lo || t < keep);
        float p[2];
#pragma unroll
        for (int mp = 0; mp < 2; mp++) {
            const T* kt = k_cache + (((size_t)page * 2 * G + 2 * g + mp) * BC_PAGE + t0 % BC_PAGE + lane) * D;
            const float s = seen ? da_dot<T>(kt, qs[warp][mp], D) * scale : -INFINITY;
            const float mn = fmaxf(m[mp], warp_max(s));
            const float corr = mn == -INFINITY ? 1.0f : expf(m[mp] - mn);
            p[mp] = seen ? expf(s - mn) : 0.0f;
            l[mp] = l[mp] * corr + warp_sum(p[mp]);
            m[mp] = mn;
#pragma unroll
            for (int j = 0; j < DA_MAX_D / 32; j++) acc[mp][j] *= corr;
        }
        const T* vt = v_cache + (((size_t)page * G + g) * BC_PAGE + t0 % BC_PAGE) * DV;
        const int n = min(32, pos + 1 - t0);
        for (int i = 0; i < n; i++) {
            if (!(t0 + i >= lo || t0 + i < keep)) continue;
            const float p0 = __shfl_sync(0xffffffffu, p[0], i), p1 = __shfl_sync(0xffffffffu, p[1], i);
#pragma unroll
            for (int j = 0; j < DA_MAX_D / 32; j++) {
                const int d = lane + 32 * j;
                if (d < DV) {
                    const float v = to_f32(vt[(size_t)i * DV + d]);
                    acc[0][j] = fmaf(p0, v, acc[0][j]);
                    acc[1][j] = fmaf(p1, v, acc[1][j]);
                }
            }
        }
    }
    const float i0 = l[0] > 0.0f ? 1.0f / l[0] : 0.0f, i1 = l[1] > 0.0f ? lambda / l[1] : 0.0f;
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < DA_MAX_D / 32; j++) {
        if (lane + 32 * j >= DV) break;
        acc[0][j] = acc[0][j] * i0 - acc[1][j] * i1;
        ss = fmaf(acc[0][j], acc[0][j], ss);
    }
    const float f = factor / sqrtf(warp_sum(ss) / (float)DV + eps);
#pragma unroll
    for (int j = 0; j < DA_MAX_D / 32; j++)
        if (lane + 32 * j < DV) o[lane + 32 * j] = from_f32<T>(acc[0][j] * f);
}

template <class T>
static int rows_launch(const void* q, const void* k_cache, const void* v_cache, const int* page_table, const int* row_pos, const int* row_slot, void* out,
                       int rows, int H, int G, int D, int DV, int max_pages, int n_pages, int window, int keep, float scale, float lambda, float eps,
                       float factor, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && G > 0 && H > 0 && H % G == 0 && (H + DA_WARPS - 1) / DA_WARPS <= 65535, "diff_rows: bad sizes rows=%d H=%d G=%d", rows, H, G);
    BC_CHECK_ARG(D > 0 && D <= DA_MAX_D && DV > 0 && DV <= DA_MAX_D && window >= 0 && keep >= 0, "diff_rows: map width %d or value width %d (1 to %d), window %d, kept %d",
                 D, DV, DA_MAX_D, window, keep);
    if (rows == 0) return BC_OK;
    bc_launch(diff_rows_kernel<T>, dim3(rows, (H + DA_WARPS - 1) / DA_WARPS), dim3(DA_WARPS * 32), 0, s, (const T*)q, (const T*)k_cache, (const T*)v_cache,
              page_table, row_pos, row_slot, (T*)out, H, G, D, DV, max_pages, n_pages, window, keep, scale, lambda, eps, factor);
    BC_LAUNCH_STATUS();
}
// q: [rows, H, 2, D]; out: [rows, H, DV]; rows whose slot is negative give zeros.
extern "C" int bc_diff_rows_f32(const void* q, const void* k_cache, const void* v_cache, const int* page_table, const int* row_pos, const int* row_slot,
                                void* out, int rows, int H, int G, int D, int DV, int max_pages, int n_pages, int window, int keep, float scale,
                                float lambda, float eps, float factor, cudaStream_t s) {
    return rows_launch<float>(q, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, keep, scale, lambda, eps, factor, s);
}
extern "C" int bc_diff_rows_bf16(const void* q, const void* k_cache, const void* v_cache, const int* page_table, const int* row_pos, const int* row_slot,
                                 void* out, int rows, int H, int G, int D, int DV, int max_pages, int n_pages, int window, int keep, float scale,
                                 float lambda, float eps, float factor, cudaStream_t s) {
    return rows_launch<bf16>(q, k_cache, v_cache, page_table, row_pos, row_slot, out, rows, H, G, D, DV, max_pages, n_pages, window, keep, scale, lambda, eps, factor, s);
}

// --------------------------------------------------------------------------------------- tiles
// Byte offset of 16-byte chunk c of row r in a [64][D] bf16 tile, chunks xor-ed so that eight rows hit eight different banks.
template <int D> __device__ __forceinline__ int da_offset(int r, int c) {
    constexpr int CHUNKS = D / 8;
    static_assert(CHUNKS == 4 || CHUNKS % 8 == 0, "tile widths are 32 or multiples of 64");
    return (r * CHUNKS + (CHUNKS == 4 ? (c ^ ((r >> 1) & 3)) : (c ^ (r & 7)))) * 16;
}

// DP, VP: map and value widths of the tiles, D and DV rounded up (what lies past the true widths is zero).  WM: warps a map, sixteen
// rows each.  With `scratch` the block takes one of gridDim.z / seqs shares of the pages and leaves its rows' parts there:
// [row][H][split][2][DV + 2] floats, products then maximum (base 2) then sum.
template <int DP, int VP, int WM, int STAGES>
__global__ void __launch_bounds__(64 * WM, WM == 1 ? 1 : VP <= 128 ? 3 : 2)
diff_tiles_kernel(const bf16* q, const bf16* k_cache, const bf16* v_cache, const int* __restrict__ page_table, const int* __restrict__ seq_rows,
                  const int* __restrict__ seq_slot, const int* __restrict__ seq_start, bf16* __restrict__ out, float* __restrict__ scratch, int splits, int H,
                  int G, int D, int DV, int max_pages, int n_pages, int window, int keep, float scale_log2, float lambda, float eps, float factor) {
    constexpr int THREADS = 64 * WM, ROWS = 16 * WM;
    constexpr int K_BYTES = 64 * DP * 2, STAGE = 2 * K_BYTES + 64 * VP * 2;
    constexpr int KD = DP / 16, ND = VP / 8;
    extern __shared__ __align__(128) uint8_t smem[];
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(q); PDL_FRESH(k_cache); PDL_FRESH(v_cache);
    const int g = blockIdx.x, sq = blockIdx.z / splits, split = blockIdx.z % splits;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int map = warp / WM, wr = warp % WM;            // which map, which sixteen rows
    const int gq = lane >> 2, tq = lane & 3;
    const int group = H / G;
    const int tokens_per_tile = ROWS / group;             // rows past tokens_per_tile * group are padding
    const int slot = seq_slot[sq];
    const int row0 = seq_rows[sq], n_new = seq_rows[sq + 1] - row0;
    const int n_tiles_q = (n_new + tokens_per_tile - 1) / tokens_per_tile;
    const int q_tile = n_tiles_q - 1 - (int)blockIdx.y;   // the tiles that see the most go first
    if (slot < 0 || q_tile < 0) return;
    const int start = seq_start[sq];
    const int tok0 = q_tile * tokens_per_tile, tok_end = min(n_new, tok0 + tokens_per_tile);
    const int* pages = page_table + (size_t)slot * max_pages;
    auto first_seen = [&](int p) { return window > 0 && p + 1 > window ? p + 1 - window : 0; };
    int tok[2], head[2], pos[2], lo[2];
    bool live[2];
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const int row = 16 * wr + gq + 8 * i;
        tok[i] = tok0 + row / group;
        head[i] = g * group + row % group;
        live[i] = row / group < tokens_per_tile && tok[i] < n_new;
        pos[i] = start + tok[i];
        lo[i] = first_seen(pos[i]);
    }
    // What all sixteen rows of the warp see: from the last row's first position (or before `keep`) to the first row's own.
    const int warp_lo = first_seen(start + tok0 + (16 * wr + 15) / group), warp_hi = start + tok0 + (16 * wr) / group;
    const bool warp_live = tok0 + (16 * wr) / group < n_new && (16 * wr) / group < tokens_per_tile;
    uint32_t qf[KD][4];
#pragma unroll
    for (int kd = 0; kd < KD; kd++) {
        const int d0 = kd * 16 + 2 * tq;
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const bf16* qr = q + (((size_t)(row0 + tok[i]) * H + head[i]) * 2 + map) * D;
            qf[kd][i] = live[i] && d0 < D ? *reinterpret_cast<const uint32_t*>(qr + d0) : 0u;
            qf[kd][i + 2] = live[i] && d0 + 8 < D ? *reinterpret_cast<const uint32_t*>(qr + d0 + 8) : 0u;
        }
    }
    const DaPages walk(start + tok0, start + tok_end - 1, window, keep);
    const int it0 = (int)((long long)walk.count * split / splits), it1 = (int)((long long)walk.count * (split + 1) / splits);
    const int last_pos = start + n_new - 1;               // the last position the sequence holds after this step
    if (D < DP || DV < VP) {
        // Columns past the true widths: no copy ever lands there.
        for (int i = threadIdx.x; i < STAGES * STAGE / 16; i += THREADS) *reinterpret_cast<uint4*>(smem + (size_t)i * 16) = make_uint4(0u, 0u, 0u, 0u);
        __syncthreads();
    }
    // A tile without a page is neither fetched nor multiplied.
    auto load = [&](int it, int stage) {
        const int tile = walk.page(it);
        const int page = tile < max_pages ? pages[tile] : -1;
        if (page < 0 || page >= n_pages) return;
        const bf16* ks = k_cache + ((size_t)page * G + g) * 2 * BC_PAGE * D;
        const bf16* vs = v_cache + ((size_t)page * G + g) * BC_PAGE * DV;
        const uint32_t kb = ad_smem(smem + (size_t)stage * STAGE), vb = kb + 2 * K_BYTES;
        const int kc = D / 8, vc = DV / 8;
        for (int i = threadIdx.x; i < 128 * kc; i += THREADS) {           // both maps: 128 rows, one after the other in the page
            const int row = i / kc, c = i - row * kc;
            cp_async16(kb + (row >> 6) * K_BYTES + da_offset<DP>(row & 63, c), ks + (size_t)row * D + c * 8);
        }
        for (int i = threadIdx.x; i < 64 * vc; i += THREADS) {
            const int row = i / vc, c = i - row * vc;
            cp_async16(vb + da_offset<VP>(row, c), vs + (size_t)row * DV + c * 8);
        }
    };
    float o[ND][4];
#pragma unroll
    for (int i = 0; i < ND; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
    for (int s = 0; s < STAGES - 1; s++) {
        if (it0 + s < it1) load(it0 + s, s);
        cp_async_commit();
    }
    const int j4 = lane >> 3, r8 = lane & 7;
    for (int it = it0; it < it1; it++) {
        const int at = (it - it0) % STAGES;
        cp_async_wait<STAGES - 2>();
        __syncthreads();
        if (it + STAGES - 1 < it1) load(it + STAGES - 1, (it - it0 + STAGES - 1) % STAGES);
        cp_async_commit();
        const int tile = walk.page(it);
        const bool page_ok = tile < max_pages && pages[tile] >= 0 && pages[tile] < n_pages;
        if (!page_ok) continue;
        const uint32_t kb = ad_smem(smem + (size_t)at * STAGE) + map * K_BYTES, vb = ad_smem(smem + (size_t)at * STAGE) + 2 * K_BYTES;
        if (tile == last_pos / BC_PAGE && last_pos % BC_PAGE != BC_PAGE - 1) {
            // What lies past the sequence's last position belongs to nobody and may be not-a-numbers: cleared in the copy.
            uint8_t* vt = smem + (size_t)at * STAGE + 2 * K_BYTES;
            const int first = last_pos % BC_PAGE + 1;
            for (int i = threadIdx.x; i < (BC_PAGE - first) * (VP / 8); i += THREADS)
                *reinterpret_cast<uint4*>(vt + da_offset<VP>(first + i / (VP / 8), i % (VP / 8))) = make_uint4(0u, 0u, 0u, 0u);
            __syncthreads();
        }
        // Nothing of this page is seen by the warp's rows (all of them are masked): the other warps alone work on it.
        const int p0 = tile * BC_PAGE;
        const int seen_from = first_seen(warp_hi), seen_to = start + min(tok_end - 1, tok0 + (16 * wr + 15) / group);
        if (!warp_live || p0 > seen_to || (p0 + BC_PAGE - 1 < seen_from && p0 >= keep)) continue;
        float s[8][4];
#pragma unroll
        for (int nb = 0; nb < 8; nb++) s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.0f;
#pragma unroll
        for (int kd = 0; kd < KD; kd++) {
#pragma unroll
            for (int np = 0; np < 4; np++) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4(kb + da_offset<DP>(np * 16 + (j4 >> 1) * 8 + r8, kd * 2 + (j4 & 1)), b0, b1, b2, b3);
                mma_16816(s[2 * np], qf[kd], b0, b1);
                mma_16816(s[2 * np + 1], qf[kd], b2, b3);
            }
        }
        float tmax[2] = {-INFINITY, -INFINITY};
        const bool whole = p0 + BC_PAGE - 1 <= warp_hi && (p0 >= warp_lo || p0 + BC_PAGE <= keep);
        if (whole) {
#pragma unroll
            for (int nb = 0; nb < 8; nb++)
#pragma unroll
                for (int e = 0; e < 4; e++) tmax[e >> 1] = fmaxf(tmax[e >> 1], s[nb][e]);
        } else {
#pragma unroll
            for (int nb = 0; nb < 8; nb++)
#pragma unroll
                for (int e = 0; e < 4; e++) {
                    const int i = e >> 1, t = p0 + nb * 8 + 2 * tq + (e & 1);
                    const bool seen = live[i] && t <= pos[i] && (t >= lo[i] || t < keep);
                    s[nb][e] = seen ? s[nb][e] : -INFINITY;
                    tmax[i] = fmaxf(tmax[i], s[nb][e]);
                }
        }
        float corr[2], base[2];
#pragma unroll
        for (int i = 0; i < 2; i++) {
            tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 1));
            tmax[i] = fmaxf(tmax[i], __shfl_xor_sync(0xffffffffu, tmax[i], 2));
            const float mn = fmaxf(m[i], tmax[i] * scale_log2);        // the scale is positive: the largest score is the largest product
            corr[i] = mn == -INFINITY ? 1.0f : fast_exp2(m[i] - mn);
            base[i] = mn == -INFINITY ? 0.0f : mn;
            m[i] = mn;
        }
        float psum[2] = {0.0f, 0.0f};
#pragma unroll
        for (int nb = 0; nb < 8; nb++)
#pragma unroll
            for (int e = 0; e < 4; e++) {
                s[nb][e] = fast_exp2(fmaf(s[nb][e], scale_log2, -base[e >> 1]));
                psum[e >> 1] += s[nb][e];
            }
        l[0] = l[0] * corr[0] + psum[0];
        l[1] = l[1] * corr[1] + psum[1];
        if (__any_sync(0xffffffffu, corr[0] != 1.0f || corr[1] != 1.0f)) {      // most pages raise no row's maximum
#pragma unroll
            for (int nd = 0; nd < ND; nd++) {
                o[nd][0] *= corr[0]; o[nd][1] *= corr[0]; o[nd][2] *= corr[1]; o[nd][3] *= corr[1];
            }
        }
#pragma unroll
        for (int kk = 0; kk < 4; kk++) {
            const uint32_t pf[4] = {pack_bf16(s[2 * kk][0], s[2 * kk][1]), pack_bf16(s[2 * kk][2], s[2 * kk][3]),
                                    pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]), pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3])};
#pragma unroll
            for (int nd = 0; nd < ND; nd += 2) {
                uint32_t b0, b1, b2, b3;
                ldmatrix_x4_trans(vb + da_offset<VP>(kk * 16 + (j4 & 1) * 8 + r8, nd + (j4 >> 1)), b0, b1, b2, b3);
                mma_16816(o[nd], pf, b0, b1);
                mma_16816(o[nd + 1], pf, b2, b3);
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int i = 0; i < 2; i++) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    }
    if (scratch != nullptr) {
#pragma unroll
        for (int i = 0; i < 2; i++) {
            if (!live[i]) continue;
            float* part = scratch + ((((size_t)(row0 + tok[i]) * H + head[i]) * splits + split) * 2 + map) * (DV + 2);
#pragma unroll
            for (int nd = 0; nd < ND; nd++) {
                const int d = nd * 8 + 2 * tq;
                if (d < DV) *reinterpret_cast<float2*>(part + d) = make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
            }
            if (tq == 0) *reinterpret_cast<float2*>(part + DV) = make_float2(m[i], l[i]);
        }
        return;
    }
    // Map 1 hands its rows over through the (now unused) page buffers, thread by thread; map 0 takes the difference, its norm and the factor.
    __syncthreads();
    float* other = reinterpret_cast<float*>(smem) + (size_t)wr * 32 * ND * 4 + lane;
    if (map == 1) {
#pragma unroll
        for (int i = 0; i < 2; i++) {
            const float inv = l[i] > 0.0f ? lambda / l[i] : 0.0f;
#pragma unroll
            for (int nd = 0; nd < ND; nd++) {
                other[(nd * 4 + 2 * i) * 32] = o[nd][2 * i] * inv;
                other[(nd * 4 + 2 * i + 1) * 32] = o[nd][2 * i + 1] * inv;
            }
        }
    }
    __syncthreads();
    if (map == 1) return;
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const float inv = l[i] > 0.0f ? 1.0f / l[i] : 0.0f;
        float ss = 0.0f;
#pragma unroll
        for (int nd = 0; nd < ND; nd++)
#pragma unroll
            for (int e = 2 * i; e < 2 * i + 2; e++) {
                o[nd][e] = o[nd][e] * inv - other[(nd * 4 + e) * 32];
                ss = fmaf(o[nd][e], o[nd][e], ss);
            }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        const float f = factor / sqrtf(ss / (float)DV + eps);
        if (!live[i]) continue;
        bf16* dst = out + ((size_t)(row0 + tok[i]) * H + head[i]) * DV + 2 * tq;
#pragma unroll
        for (int nd = 0; nd < ND; nd++)
            if (nd * 8 + 2 * tq < DV) *reinterpret_cast<uint32_t*>(dst + nd * 8) = pack_bf16(o[nd][2 * i] * f, o[nd][2 * i + 1] * f);
    }
}

// The splits' parts of a (row, head), added up in their order; both maps, then the difference, its norm and the factor.
__global__ void __launch_bounds__(128)
diff_merge_kernel(const float* scratch, const int* __restrict__ row_slot, bf16* __restrict__ out, int H, int DV, int splits, float lambda, float eps,
                  float factor) {
    __shared__ float red[32];
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(scratch);
    const int r = blockIdx.x, h = blockIdx.y;
    bf16* o = out + ((size_t)r * H + h) * DV;
    if (row_slot[r] < 0) {
        for (int d = threadIdx.x; d < DV; d += blockDim.x) o[d] = __float2bfloat16_rn(0.0f);
        return;
    }
    const float* parts = scratch + ((size_t)r * H + h) * splits * 2 * (DV + 2);
    float top[2] = {-INFINITY, -INFINITY}, sum[2] = {0.0f, 0.0f};
    for (int s = 0; s < splits; s++)
#pragma unroll
        for (int mp = 0; mp < 2; mp++) top[mp] = fmaxf(top[mp], parts[(size_t)(2 * s + mp) * (DV + 2) + DV]);
    for (int s = 0; s < splits; s++)
#pragma unroll
        for (int mp = 0; mp < 2; mp++) {
            const float* ml = parts + (size_t)(2 * s + mp) * (DV + 2) + DV;
            if (ml[0] != -INFINITY) sum[mp] += ml[1] * fast_exp2(ml[0] - top[mp]);
        }
    float z[2], ss = 0.0f;
#pragma unroll
    for (int j = 0; j < 2; j++) {
        const int d = threadIdx.x + j * 128;
        z[j] = 0.0f;
        if (d >= DV) continue;
        float a[2] = {0.0f, 0.0f};
        for (int s = 0; s < splits; s++)
#pragma unroll
            for (int mp = 0; mp < 2; mp++) {
                const float* p = parts + (size_t)(2 * s + mp) * (DV + 2);
                if (p[DV] != -INFINITY) a[mp] = fmaf(p[d], fast_exp2(p[DV] - top[mp]), a[mp]);
            }
        z[j] = (sum[0] > 0.0f ? a[0] / sum[0] : 0.0f) - lambda * (sum[1] > 0.0f ? a[1] / sum[1] : 0.0f);
        ss = fmaf(z[j], z[j], ss);
    }
    const float f = factor / sqrtf(block_sum(ss, red) / (float)DV + eps);
#pragma unroll
    for (int j = 0; j < 2; j++) {
        const int d = threadIdx.x + j * 128;
        if (d < DV) o[d] = __float2bfloat16_rn(z[j] * f);
    }
}

template <int DP, int VP, int WM>
static int tiles_launch(const void* q, const void* k_cache, const void* v_cache, const int* page_table, const int* seq_rows, const int* seq_slot,
                        const int* seq_start, void* out, float* scratch, int splits, int seqs, int max_new, int H, int G, int D, int DV, int max_pages,
                        int n_pages, int window, int keep, float scale, float lambda, float eps, float factor, cudaStream_t s) {
    constexpr int STAGE = 64 * (2 * DP + VP) * 2;
    constexpr int STAGES = WM == 1 && 3 * STAGE <= 110 * 1024 ? 3 : 2;      // few rows: more bytes on their way
    constexpr int SMEM = STAGES * STAGE;
    static_assert(SMEM >= WM * 32 * (VP / 8) * 4 * 4, "the maps meet in the page buffers");
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(diff_tiles_kernel<DP, VP, WM, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) {
            bc_set_error("diff_tiles: cannot set shared memory to %d: %s", SMEM, cudaGetErrorString(e));
            return (int)e;
        }
        configured = true;
    }
    const int tokens_per_tile = 16 * WM / (H / G);
    dim3 grid(G, (max_new + tokens_per_tile - 1) / tokens_per_tile, seqs * splits);
    cudaError_t e = bc_launch(diff_tiles_kernel<DP, VP, WM, STAGES>, grid, dim3(64 * WM), (size_t)SMEM, s, (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache,
                              page_table, seq_rows, seq_slot, seq_start, (bf16*)out, scratch, splits, H, G, D, DV, max_pages, n_pages, window, keep,
                              scale * 1.4426950408889634f, lambda, eps, factor);
    if (e != cudaSuccess) {
        bc_set_error("diff_tiles: %s", cudaGetErrorString(e));
        return (int)e;
    }
    BC_LAUNCH_STATUS();
}

// Whether the tile kernel takes the sizes (else the rows kernel serves): widths multiples of 8, maps up to 128, values up to 256, at
// most 32 heads a kv head.
extern "C" int bc_diff_tiles_accepts(int H, int G, int D, int DV) {
    return G > 0 && H % G == 0 && H / G <= 32 && D % 8 == 0 && D > 0 && D <= 128 && DV % 8 == 0 && DV > 0 && DV <= 256;
}

// q: [rows, H, 2, D] bf16; out: [rows, H, DV]; sequence s owns rows seq_rows[s] .. seq_rows[s + 1], lives in slot seq_slot[s] (negative:
// skipped, its rows of `out` are left untouched) and held seq_start[s] positions before this step; the cache already holds this step's
// keys and values.  splits > 1: scratch holds rows * H * splits * 2 * (DV + 2) floats and row_slot [rows] marks padding rows.
extern "C" int bc_diff_tiles_bf16(const void* q, const void* k_cache, const void* v_cache, const int* page_table, const int* seq_rows, const int* seq_slot,
                                  const int* seq_start, const int* row_slot, void* out, float* scratch, int splits, int rows, int seqs, int max_new, int H,
                                  int G, int D, int DV, int max_pages, int n_pages, int window, int keep, float scale, float lambda, float eps, float factor,
                                  cudaStream_t s) {
    BC_CHECK_ARG(bc_diff_tiles_accepts(H, G, D, DV), "diff_tiles: H=%d G=%d D=%d DV=%d is outside what this kernel takes", H, G, D, DV);
    BC_CHECK_ARG(seqs >= 0 && splits >= 1 && (long long)seqs * splits <= 65535 && max_new >= 0 && max_new < 65535, "diff_tiles: bad sizes seqs=%d splits=%d max_new=%d",
                 seqs, splits, max_new);
    BC_CHECK_ARG(scale > 0.0f, "diff_tiles: a scale of %g is not positive", (double)scale);
    BC_CHECK_ARG(window >= 0 && keep >= 0 && (splits == 1 || (scratch && row_slot)), "diff_tiles: bad window %d, kept %d or no scratch", window, keep);
    BC_CHECK_ARG((uintptr_t)q % 4 == 0 && (uintptr_t)out % 4 == 0 && (uintptr_t)k_cache % 16 == 0 && (uintptr_t)v_cache % 16 == 0, "diff_tiles: unaligned operands");
    if (seqs == 0 || max_new == 0) return BC_OK;
    int st = BC_ERR_ARG;
    const bool few = (long long)max_new * (H / G) <= 16;
#define DA_GO(DP_, VP_, WM_)                                                                                                                            \
    st = tiles_launch<DP_, VP_, WM_>(q, k_cache, v_cache, page_table, seq_rows, seq_slot, seq_start, out, splits > 1 ? scratch : nullptr, splits, seqs, max_new, H, \
                                     G, D, DV, max_pages, n_pages, window, keep, scale, lambda, eps, factor, s)
#define DA_V(DP_, VP_)                    \
    do {                                  \
        if (few) DA_GO(DP_, VP_, 1);      \
        else DA_GO(DP_, VP_, 2);          \
    } while (0)
#define DA_D(DP_)                         \
    do {                                  \
        if (DV <= 32) DA_V(DP_, 32);      \
        else if (DV <= 64) DA_V(DP_, 64); \
        else if (DV <= 128) DA_V(DP_, 128); \
        else if (DV <= 192) DA_V(DP_, 192); \
        else DA_V(DP_, 256);              \
    } while (0)
    if (D <= 32) DA_D(32);
    else if (D <= 64) DA_D(64);
    else DA_D(128);
#undef DA_D
#undef DA_V
#undef DA_GO
    if (st != BC_OK || splits == 1) return st;
    bc_launch(diff_merge_kernel, dim3(rows, H), dim3(128), 0, s, (const float*)scratch, row_slot, (bf16*)out, H, DV, splits, lambda, eps, factor);
    BC_LAUNCH_STATUS();
}
