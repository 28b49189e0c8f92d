// Differential attention for prompts on the 5th-generation tensor cores (bf16, maps of 64 or 128, values of 64 or 128).
//
// What is computed is diff_attention.cu's.  A block takes ONE tile of 128 query rows = (tokens) x (the heads that share the kv
// head), token major, of one sequence, and both maps of it: what attention_prefill_tc.cu does with two tiles of query rows on one
// key, this kernel does with the two maps of one tile on their two keys, so a page's two key maps and its values are fetched once:
//
//   - queries come by one 3-d TMA box a map and 64 elements out of [row][head][map][d], a page by 2-d boxes (both key maps, values)
//     into a ring of stages;
//   - S_m = Q_m K_m^T (tcgen05.mma, M 128, N 64 positions) into two score buffers a map in TMEM; four softmax warps a map, one row a
//     thread, mask, exponentiate and write P back over the scores it came from;
//   - O_m += P_m V with A out of tensor memory and the values as the n-major B operand both maps share;
//   - at the end both accumulators lie in the same TMEM lanes: the thread of row r of map m takes half of the row's value columns,
//     A_0 - lambda A_1, the row's sum of squares meets in shared memory, and the normed row is rounded once.
//
// Masks: causal, a sliding window that keeps a sequence's first positions (pages between the two are skipped), ragged sequences,
// continuation from cached positions.  Warp roles: warp 0 issues TMA, warp 1 owns TMEM and issues the MMAs, warps 2-5 are the softmax
// of map 0 and warps 6-9 of map 1.  Every wait is bounded (about a second); a wait that gives up records where in a status word,
// and the block frees its TMEM and returns.
#include "mma_tiles.cuh"
#include "tc_ptx.cuh"
#include "tma_host.cuh"

#define DT_ROWS 128
#define DT_THREADS 320
#define DT_PAGES_KEPT 256
#define DT_SMEM_LIMIT 232448
#define DT_Q_BYTES(D) (2 * ((D) / 64) * DT_ROWS * 128)
#define DT_STAGE_BYTES(D, DV) ((2 * ((D) / 64) + (DV) / 64) * 64 * 128)
#define DT_STAGES_FIT(D, DV) ((DT_SMEM_LIMIT - 4096 - DT_Q_BYTES(D)) / DT_STAGE_BYTES(D, DV))
#define DT_STAGES(D, DV) (DT_STAGES_FIT(D, DV) > 6 ? 6 : DT_STAGES_FIT(D, DV))
#define DT_RAISE 8.0f       // the running maximum follows the true one at this distance at most (log2 units)

template <int D, int DV>
__global__ void __launch_bounds__(DT_THREADS, 1)
diff_attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                         const int* __restrict__ page_table, const int* __restrict__ seq_rows, const int* __restrict__ seq_slot,
                         const int* __restrict__ seq_start, bf16* __restrict__ out, int H, int G, int max_pages, int n_pages, int window, int keep,
                         float scale_log2, float lambda, float eps, float factor) {
    constexpr int STAGES = DT_STAGES(D, DV);
    constexpr int DB = D / 64, DVB = DV / 64;
    constexpr int ROW_BLOCK = DT_ROWS * 128;           // bytes of a [128 rows][64 elements] block
    constexpr int KV_BLOCK = BC_PAGE * 128;            // bytes of a [64 positions][64 elements] block
    constexpr int STAGE_BYTES = DT_STAGE_BYTES(D, DV); // keys of map 0, keys of map 1, values
    constexpr int V_AT = 2 * DB * KV_BLOCK;
    constexpr int O_COL = 256;                         // TMEM columns: scores of (map m, buffer b) from (2 m + b) 64, outputs from O_COL + m DV
    static_assert(STAGES >= 2, "the ring does not fit");
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    uint8_t* smem = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    uint8_t* q_smem = smem;                            // map m, block b at (m DB + b) ROW_BLOCK
    uint8_t* kv_smem = q_smem + DT_Q_BYTES(D);
    __shared__ __align__(8) uint64_t bars[2 * STAGES + 1 + 12];
    __shared__ uint32_t tmem_slot;
    __shared__ int page_of[DT_PAGES_KEPT];             // the first pages this block reads, fetched once (-1: none)
    __shared__ float row_sum[2][DT_ROWS], row_ss[2][DT_ROWS];

    pdl_launch_dependents();
    pdl_wait();
    const int g = blockIdx.x, sq = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int group = H / G;
    const int tokens_per_block = DT_ROWS / group;      // rows past tokens_per_block * group are padding
    const int slot = seq_slot[sq];
    const int row0 = seq_rows[sq], n_new = seq_rows[sq + 1] - row0;
    const int n_blocks_q = (n_new + tokens_per_block - 1) / tokens_per_block;
    const int q_block = n_blocks_q - 1 - (int)blockIdx.y;      // the rows that see the most go first
    if (slot < 0 || q_block < 0) return;                       // the whole block, before anything is set up
    const int start = seq_start[sq];
    const int tok0 = q_block * tokens_per_block;
    const int tok_end = min(n_new, tok0 + tokens_per_block);
    const int* pages = page_table + (size_t)slot * max_pages;
    // Pages this block reads, in order: those of the kept first positions, then those from the oldest position its first token's window shows.
    const int first_pos = window > 0 && start + tok0 + 1 > window ? start + tok0 + 1 - window : 0;
    const int first_page = first_pos / BC_PAGE, kept = min(first_page, (keep + BC_PAGE - 1) / BC_PAGE);
    const int n_tiles = kept + (start + tok_end - 1) / BC_PAGE + 1 - first_page;
    auto tile_at = [&](int j) { return j < kept ? j : first_page + (j - kept); };
    const int last_pos = start + n_new - 1;

    const uint32_t kv_full0 = smem_u32(&bars[0]), kv_empty0 = smem_u32(&bars[STAGES]), q_full = smem_u32(&bars[2 * STAGES]);
    // Per map and buffer: scores ready, P written, product done.
    auto s_full = [&](int m, int b) { return smem_u32(&bars[2 * STAGES + 1 + 6 * m + b]); };
    auto p_full = [&](int m, int b) { return smem_u32(&bars[2 * STAGES + 1 + 6 * m + 2 + b]); };
    auto o_done = [&](int m, int b) { return smem_u32(&bars[2 * STAGES + 1 + 6 * m + 4 + b]); };
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            mbar_init(kv_full0 + 8 * s, 1);
            mbar_init(kv_empty0 + 8 * s, 1);
        }
        mbar_init(q_full, 1);
        for (int m = 0; m < 2; m++)
            for (int b = 0; b < 2; b++) {
                mbar_init(s_full(m, b), 1);
                mbar_init(p_full(m, b), 128);
                mbar_init(o_done(m, b), 1);
            }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(smem_u32(&tmem_slot), 512);
    for (int i = threadIdx.x; i < min(n_tiles, DT_PAGES_KEPT); i += DT_THREADS) {
        const int tile = tile_at(i);
        const int page = tile < max_pages ? pages[tile] : -1;
        page_of[i] = page >= 0 && page < n_pages ? page : -1;
    }
    auto page_at = [&](int j) {
        if (j < DT_PAGES_KEPT) return page_of[j];
        const int tile = tile_at(j);
        const int page = tile < max_pages ? pages[tile] : -1;
        return page >= 0 && page < n_pages ? page : -1;
    };
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = tmem_slot;

    if (warp == 0) {
        if (lane == 0) {
            mbar_expect_tx(q_full, (uint32_t)(2 * DB * tokens_per_block * group * 128));
            for (int m = 0; m < 2; m++)
                for (int b = 0; b < DB; b++) tma_load_3d(smem_u32(q_smem + (m * DB + b) * ROW_BLOCK), &map_q, q_full, m * D + b * 64, g * group, row0 + tok0);
            for (int j = 0; j < n_tiles; j++) {
                const int s = j % STAGES;
                if (j >= STAGES && !mbar_wait(kv_empty0 + 8 * s, ((j / STAGES) & 1) ^ 1, 1)) break;
                const int page = page_at(j);
                if (page < 0) {
                    // No page: nothing is fetched; the scores of whatever the stage still holds are masked, its values cleared before use.
                    mbar_arrive(kv_full0 + 8 * s);
                    continue;
                }
                const uint32_t dst = smem_u32(kv_smem + (size_t)s * STAGE_BYTES);
                mbar_expect_tx(kv_full0 + 8 * s, STAGE_BYTES);
                for (int m = 0; m < 2; m++)
                    for (int b = 0; b < DB; b++)
                        tma_load_2d(dst + (m * DB + b) * KV_BLOCK, &map_k, kv_full0 + 8 * s, b * 64, ((page * G + g) * 2 + m) * BC_PAGE);
                for (int b = 0; b < DVB; b++) tma_load_2d(dst + V_AT + b * KV_BLOCK, &map_v, kv_full0 + 8 * s, b * 64, (page * G + g) * BC_PAGE);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc_s = instr_desc_b(BC_PAGE, false);   // S: N = 64 positions, keys k-major
            constexpr uint32_t idesc_o = instr_desc_b(DV, true);         // O: N = the values' width, values n-major
            const uint64_t q_desc0 = smem_desc(smem_u32(q_smem));
            const uint64_t k_desc0 = smem_desc(smem_u32(kv_smem));
            const uint64_t v_desc0 = smem_desc_mn(smem_u32(kv_smem) + V_AT, KV_BLOCK);
            auto scores = [&](int j) {
                const uint64_t k_desc = k_desc0 + (uint64_t)((j % STAGES) * (STAGE_BYTES >> 4));
#pragma unroll
                for (int m = 0; m < 2; m++) {
#pragma unroll
                    for (int kk = 0; kk < D / 16; kk++)
                        mma_bf16(tmem + (2 * m + (j & 1)) * BC_PAGE, q_desc0 + (uint64_t)(((m * DB + (kk >> 2)) * ROW_BLOCK >> 4) + 2 * (kk & 3)),
                                 k_desc + (uint64_t)(((m * DB + (kk >> 2)) * KV_BLOCK >> 4) + 2 * (kk & 3)), idesc_s, kk != 0);
                    mma_commit(s_full(m, j & 1));
                }
            };
            bool ok = mbar_wait(q_full, 0, 2);
            for (int j = 0; j < 2 && j < n_tiles && ok; j++) {
                ok = mbar_wait(kv_full0 + 8 * (j % STAGES), 0, 3);
                if (!ok) break;
                tc_fence_after();
                scores(j);
            }
            for (int j = 0; j < n_tiles && ok; j++) {
                const uint64_t v_desc = v_desc0 + (uint64_t)((j % STAGES) * (STAGE_BYTES >> 4));   // 16 positions on: 2048 bytes
#pragma unroll
                for (int m = 0; m < 2; m++) {
                    ok = ok && mbar_wait(p_full(m, j & 1), (j >> 1) & 1, 4);
                    if (!ok) break;
                    tc_fence_after();
                    // P lies over the first 32 columns of the scores it came from: 8 columns a k-step of 16 positions.
#pragma unroll
                    for (int kk = 0; kk < BC_PAGE / 16; kk++)
                        mma_bf16_a_tmem(tmem + O_COL + m * DV, tmem + (2 * m + (j & 1)) * BC_PAGE + 8 * kk, v_desc + (uint64_t)(kk * (2048 >> 4)), idesc_o,
                                        (j | kk) != 0);
                    mma_commit(o_done(m, j & 1));
                }
                if (!ok) break;
                mma_commit(kv_empty0 + 8 * (j % STAGES));
                if (j + 2 < n_tiles) {
                    const int s = (j + 2) % STAGES;
                    ok = mbar_wait(kv_full0 + 8 * s, ((j + 2) / STAGES) & 1, 5);
                    if (!ok) break;
                    tc_fence_after();
                    scores(j + 2);
                }
            }
        }
    } else {
        const int q = warp & 3, m = (warp - 2) >> 2;
        const int row = 32 * q + lane;                                   // of the tile, and the TMEM lane
        const int tok = tok0 + row / group, head = g * group + row % group;
        const bool live = row / group < tokens_per_block && tok < n_new;
        const int pos = start + tok;
        const int lo = window > 0 && pos + 1 > window ? pos + 1 - window : 0;
        // What every row of this warp sees: from the last row's window (or before `keep`) to the first row's own position.
        const int warp_first_pos = start + tok0 + (32 * q) / group, warp_last_pos = start + tok0 + (32 * q + 31) / group;
        const int warp_lo = window > 0 && warp_last_pos + 1 > window ? warp_last_pos + 1 - window : 0;
        const uint32_t lane_base = tmem + ((uint32_t)(32 * q) << 16);
        const uint32_t o_addr = lane_base + O_COL + m * DV;
        float m_used = -INFINITY, l = 0.0f;
        bool ok = true;
        for (int j = 0; j < n_tiles; j++) {
            if (lane == 0) ok = mbar_wait(s_full(m, j & 1), (j >> 1) & 1, 6);
            ok = __shfl_sync(0xffffffffu, ok, 0);
            if (!ok) break;
            tc_fence_after();
            uint32_t sv[64];
#pragma unroll
            for (int c = 0; c < 4; c++) tmem_load16(lane_base + (2 * m + (j & 1)) * BC_PAGE + 16 * c, sv + 16 * c);
            tmem_load_wait();
            const int p0 = tile_at(j) * BC_PAGE;
            const bool page_ok = page_at(j) >= 0;
            const bool whole = page_ok && p0 + BC_PAGE - 1 <= warp_first_pos && (p0 >= warp_lo || p0 + BC_PAGE <= keep);
            float tmax = -INFINITY;
            if (whole) {
                float ta = -INFINITY, tb = -INFINITY;
#pragma unroll
                for (int c = 0; c < 64; c += 4) {
                    ta = max3(ta, __uint_as_float(sv[c]), __uint_as_float(sv[c + 1]));
                    tb = max3(tb, __uint_as_float(sv[c + 2]), __uint_as_float(sv[c + 3]));
                }
                tmax = fmaxf(ta, tb);
            } else {
#pragma unroll
                for (int c = 0; c < 64; c++) {
                    const int kpos = p0 + c;
                    const bool seen = page_ok && live && kpos <= pos && (kpos >= lo || kpos < keep);
                    const float v = seen ? __uint_as_float(sv[c]) : -INFINITY;
                    sv[c] = __float_as_uint(v);
                    tmax = fmaxf(tmax, v);
                }
            }
            const float m_true = fmaxf(m_used, tmax * scale_log2);
            const bool raise = m_true > m_used + DT_RAISE;     // also the first finite maximum: -inf + 8 = -inf
            float corr = 1.0f;
            if (raise) {
                corr = m_used == -INFINITY ? 0.0f : exp2f(m_used - m_true);
                m_used = m_true;
                l *= corr;
            }
            if (j >= 2) {
                // P goes over the scores of the page two before, whose product has to be done; waiting for every phase in order keeps
                // the parities apart.
                if (lane == 0) ok = mbar_wait(o_done(m, j & 1), ((j - 2) >> 1) & 1, 7);
                ok = __shfl_sync(0xffffffffu, ok, 0);
                if (!ok) break;
            }
            if (j > 0 && __any_sync(0xffffffffu, raise)) {
                // Rescale this warp's rows of the accumulator, once every product issued so far is in it.
                if (lane == 0) ok = mbar_wait(o_done(m, (j - 1) & 1), ((j - 1) >> 1) & 1, 9);
                ok = __shfl_sync(0xffffffffu, ok, 0);
                if (!ok) break;
                tc_fence_after();
#pragma unroll 1
                for (int c = 0; c < DV; c += 16) {
                    uint32_t ov[16];
                    tmem_load16(o_addr + c, ov);
                    tmem_load_wait();
#pragma unroll
                    for (int i = 0; i < 16; i++) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * corr);
                    tmem_store16(o_addr + c, ov);
                }
                tmem_store_wait();
            }
            const float base = m_used == -INFINITY ? 0.0f : m_used;
            const uint64_t scale2 = pack_f32x2(scale_log2, scale_log2), shift2 = pack_f32x2(-base, -base);
            uint64_t sums[4] = {0ull, 0ull, 0ull, 0ull};
            const uint32_t p_addr = lane_base + (2 * m + (j & 1)) * BC_PAGE;
#pragma unroll
            for (int c16 = 0; c16 < 2; c16++) {
                uint32_t packed[16];
#pragma unroll
                for (int i = 0; i < 16; i++) {
                    float a, b;
                    unpack_f32x2(fma_f32x2(pack_f32x2(__uint_as_float(sv[c16 * 32 + 2 * i]), __uint_as_float(sv[c16 * 32 + 2 * i + 1])), scale2, shift2), a, b);
                    a = fast_exp2(a), b = fast_exp2(b);
                    sums[i & 3] = add_f32x2(sums[i & 3], pack_f32x2(a, b));
                    packed[i] = pack_bf16(a, b);
                }
                tmem_store16(p_addr + 16 * c16, packed);
            }
            {
                float s0, s1, s2, s3;
                unpack_f32x2(add_f32x2(sums[0], sums[1]), s0, s1);
                unpack_f32x2(add_f32x2(sums[2], sums[3]), s2, s3);
                l += (s0 + s1) + (s2 + s3);
            }
            // Value rows that hold no position of this sequence (the whole page if there is none, else what lies past its last position) are
            // cleared in the copy by the threads of map 0, whose product of this page is issued first.
            const int first_bad = !page_ok ? 0 : min(BC_PAGE, max(0, last_pos - p0 + 1));
            if (m == 0 && first_bad < BC_PAGE) {
                uint8_t* v_tile = kv_smem + (size_t)(j % STAGES) * STAGE_BYTES + V_AT;
                for (int c = row; c < (BC_PAGE - first_bad) * DVB * 8; c += 128) {
                    const int vrow = first_bad + c / (DVB * 8), within = c % (DVB * 8);
                    *reinterpret_cast<uint4*>(v_tile + (within >> 3) * KV_BLOCK + vrow * 128 + (within & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
                }
                fence_proxy_async();
            }
            tmem_store_wait();
            tc_fence_before();
            mbar_arrive(p_full(m, j & 1));
        }
        if (ok) {
            if (lane == 0) ok = mbar_wait(o_done(m, (n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1, 8);
            ok = __shfl_sync(0xffffffffu, ok, 0);
        }
        // Both maps' accumulators are whole once every softmax warp has seen its own: a row's sums are exchanged at the same barrier.
        row_sum[m][row] = l;
        tc_fence_before();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        tc_fence_after();
        const float l0 = row_sum[0][row], l1 = row_sum[1][row];
        const float i0 = l0 > 0.0f ? 1.0f / l0 : 0.0f, i1 = l1 > 0.0f ? lambda / l1 : 0.0f;
        constexpr int HALF = DV / 2;
        float z[HALF], ss = 0.0f;
#pragma unroll
        for (int c = 0; c < HALF; c += 16) {
            uint32_t va[16], vb[16];
            tmem_load16(lane_base + O_COL + m * HALF + c, va);
            tmem_load16(lane_base + O_COL + DV + m * HALF + c, vb);
            tmem_load_wait();
#pragma unroll
            for (int i = 0; i < 16; i++) {
                z[c + i] = fmaf(__uint_as_float(va[i]), i0, -__uint_as_float(vb[i]) * i1);
                ss = fmaf(z[c + i], z[c + i], ss);
            }
        }
        row_ss[m][row] = ss;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        if (ok && live) {
            const float f = factor / sqrtf((row_ss[0][row] + row_ss[1][row]) / (float)DV + eps);
            bf16* dst = out + ((size_t)(row0 + tok) * H + head) * DV + m * HALF;
#pragma unroll
            for (int c = 0; c < HALF; c += 8)
                *reinterpret_cast<uint4*>(dst + c) = make_uint4(pack_bf16(z[c] * f, z[c + 1] * f), pack_bf16(z[c + 2] * f, z[c + 3] * f),
                                                                pack_bf16(z[c + 4] * f, z[c + 5] * f), pack_bf16(z[c + 6] * f, z[c + 7] * f));
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, 512);
    }
}

// -------------------------------------------------------------------------------- the host
// The queries [rows][H][2][D] as a tensor of rows of heads of 2 D elements, cut into boxes of [tokens][heads of a group][64].
static int query_map(CUtensorMap* map, const void* q, int total_rows, int H, int D, int group, int tokens) {
    cuuint64_t dims[3] = {(cuuint64_t)(2 * D), (cuuint64_t)H, (cuuint64_t)total_rows};
    cuuint64_t strides[2] = {(cuuint64_t)D * 4, (cuuint64_t)H * D * 4};
    cuuint32_t box[3] = {64, (cuuint32_t)group, (cuuint32_t)tokens};
    cuuint32_t elem[3] = {1, 1, 1};
    CUresult r = bc_encode_tiled_fn()(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, elem, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                      CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) {
        bc_set_error("diff_attention_tc: cuTensorMapEncodeTiled failed (%d) for queries [%d, %d, %d]", (int)r, total_rows, H, 2 * D);
        return BC_ERR_DRIVER;
    }
    return BC_OK;
}

template <int D, int DV>
static int launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const int* page_table, const int* seq_rows, const int* seq_slot,
                  const int* seq_start, void* out, int seqs, int max_new, int H, int G, int max_pages, int n_pages, int window, int keep, float scale, float lambda,
                  float eps, float factor, cudaStream_t s) {
    constexpr int SMEM = DT_Q_BYTES(D) + DT_STAGES(D, DV) * DT_STAGE_BYTES(D, DV) + 1024;
    static_assert(SMEM + 4096 <= DT_SMEM_LIMIT + 1024, "the ring does not fit");
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(diff_attention_tc_kernel<D, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
        if (e != cudaSuccess) {
            bc_set_error("diff_attention_tc: cannot set shared memory to %d: %s", SMEM, cudaGetErrorString(e));
            return (int)e;
        }
        configured = true;
    }
    const int tokens = DT_ROWS / (H / G);
    dim3 grid(G, (max_new + tokens - 1) / tokens, seqs);
    cudaError_t e = bc_launch(diff_attention_tc_kernel<D, DV>, grid, dim3(DT_THREADS), (size_t)SMEM, s, mq, mk, mv, page_table, seq_rows, seq_slot, seq_start,
                              (bf16*)out, H, G, max_pages, n_pages, window, keep, scale * 1.4426950408889634f, lambda, eps, factor);
    if (e != cudaSuccess) {
        bc_set_error("diff_attention_tc: launch failed: %s", cudaGetErrorString(e));
        return (int)e;
    }
    BC_LAUNCH_STATUS();
}

// Maps of 64 or 128, values of 64 or 128, at most 128 heads a kv head.
extern "C" int bc_diff_attention_tc_accepts(int H, int G, int D, int DV) {
    return G > 0 && H % G == 0 && H / G <= DT_ROWS && (D == 64 || D == 128) && (DV == 64 || DV == 128) && bc_encode_tiled_fn() != nullptr;
}

// As bc_diff_tiles_bf16 without splits; total_rows: how many rows q has in all (TMA reads past them as zeros).
extern "C" int bc_diff_attention_tc_bf16(const void* q, int total_rows, const void* k_cache, const void* v_cache, const int* page_table, const int* seq_rows,
                                         const int* seq_slot, const int* seq_start, void* out, int seqs, int max_new, int H, int G, int D, int DV, int max_pages,
                                         int n_pages, int window, int keep, float scale, float lambda, float eps, float factor, cudaStream_t s) {
    BC_CHECK_ARG(bc_diff_attention_tc_accepts(H, G, D, DV), "diff_attention_tc: H=%d G=%d D=%d DV=%d is outside what this kernel takes", H, G, D, DV);
    BC_CHECK_ARG(seqs >= 0 && seqs <= 65535 && max_new >= 0 && total_rows >= 0 && max_new / (DT_ROWS / (H / G)) < 65535, "diff_attention_tc: bad sizes seqs=%d max_new=%d rows=%d",
                 seqs, max_new, total_rows);
    BC_CHECK_ARG((uintptr_t)q % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)k_cache % 16 == 0 && (uintptr_t)v_cache % 16 == 0, "diff_attention_tc: unaligned operands");
    BC_CHECK_ARG(window >= 0 && keep >= 0 && n_pages > 0 && scale > 0.0f, "diff_attention_tc: bad window %d, kept %d, pages %d or scale %g", window, keep, n_pages, (double)scale);
    if (seqs == 0 || max_new == 0 || total_rows == 0) return BC_OK;
    CUtensorMap mq, mk, mv;
    int st = query_map(&mq, q, total_rows, H, D, H / G, DT_ROWS / (H / G));
    if (st != BC_OK) return st;
    if ((st = bc_cached_cache_map(&mk, k_cache, (long long)n_pages * 2 * G * BC_PAGE, D, "diff_attention_tc")) != BC_OK) return st;
    if ((st = bc_cached_cache_map(&mv, v_cache, (long long)n_pages * G * BC_PAGE, DV, "diff_attention_tc")) != BC_OK) return st;
#define DT_GO(DD, VV) return launch<DD, VV>(mq, mk, mv, page_table, seq_rows, seq_slot, seq_start, out, seqs, max_new, H, G, max_pages, n_pages, window, keep, scale, lambda, eps, factor, s)
    if (D == 64 && DV == 64) DT_GO(64, 64);
    if (D == 64) DT_GO(64, 128);
    if (DV == 64) DT_GO(128, 64);
    DT_GO(128, 128);
#undef DT_GO
}

TC_STATUS_EXPORTS(diff_attention_tc)
