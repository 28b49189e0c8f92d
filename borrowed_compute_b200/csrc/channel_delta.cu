// The gated delta rule with a decay a key channel: a recurrent mixer whose state is one [D, P] matrix a head (key channel i,
// value channel j) in float, carried from token to token:
//
//   S <- diag(c) S;   r = b (v - S^T k);   S <- S + k r^T;   o = S^T q        (the read-out sees the token's own write)
//
// with k and q unit vectors a head (q also over sqrt(D)), b a number a head in (0, 1) and c = exp(-exp(A) softplus(z + t)) a key
// channel, z a low-rank projection.  `rep` neighbouring heads share one q and k.  Kernels:
//
//   split    the inner vectors of low-rank projections, columns of the fused projection, as rows of their own: floats as they
//            are, or (bf16) as two terms hi + lo side by side, whose product with the outer matrix stored twice on the tensor
//            cores is then exact to about 2^-17
//   prepare  (eight rows, head) a block: decays from z; unit q and k in place of the convolved ones; b and q . k
//   scan     (sequence, head, 32 value channels) a block walks the rows of the step in time order.  A value channel j is
//            independent of the others:  with s the old column and w = c s,
//               r = b (v - k . w),   s' = w + k r,   o = q . w + (q . k) r,
//            so one pass over the old column gives both sums.  Eight threads share a column (two columns a thread), their sums
//            meet by shuffles; q, k and decays of sixteen rows at a time (fewer for wide heads) are staged in shared memory by
//            asynchronous copies, the next lot on its way while this one is walked
//   step     a step of one row a sequence: the outer products of the decay and of the output's gate, unit vectors, one step of
//            the recurrence, and the norm and gate of the head's output in one launch, a block a (row, head)
//
// Everything here is float whatever the activation type is; only the step's output takes that type.  What a thread adds and in
// which order depends on the sizes alone, never on where a prompt was cut or what else is in the batch.
#include "common.cuh"

#define CD_LANES 8          // threads that share one value channel
#define CD_COLS 16          // threads-of-eight a block of the scan
#define CD_CJ 2             // value channels a thread of the scan
#define CD_BLOCK_COLS (CD_COLS * CD_CJ)
#define CD_MAX_D 256
#define CD_ROWS 8           // rows a block of prepare
#define CD_UNIT_EPS 1e-6f

__device__ __forceinline__ float cd_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float cd_softplus(float x) { return fmaxf(x, 0.0f) + log1pf(expf(-fabsf(x))); }

// A thread's R key channels: runs of four neighbours, the eight threads' runs side by side, the next runs 32 channels on (heads of
// at most 16 channels: two neighbours a thread), so that a load of 16 bytes a thread covers 128 bytes without a gap.
template <int R> __device__ __forceinline__ int cd_channel(int lane, int q) { return R >= 4 ? (q >> 2) * 32 + lane * 4 + (q & 3) : lane * R + q; }
template <int R> __device__ __forceinline__ void cd_load(const float* vec, int lane, float* v) {
    if constexpr (R >= 4) {
#pragma unroll
        for (int m = 0; m < R / 4; m++) {
            const float4 x = *reinterpret_cast<const float4*>(vec + m * 32 + lane * 4);
            v[4 * m] = x.x; v[4 * m + 1] = x.y; v[4 * m + 2] = x.z; v[4 * m + 3] = x.w;
        }
    } else {
#pragma unroll
        for (int q = 0; q < R; q++) v[q] = vec[lane * R + q];
    }
}
template <int R> __device__ __forceinline__ void cd_load_column(const float* col, int lane, int D, bool ok, float* s) {
    if constexpr (R >= 4) {
        if (D % 4 == 0) {
#pragma unroll
            for (int q = 0; q < R; q += 4) {
                const int i = cd_channel<R>(lane, q);
                const float4 v = ok && i < D ? *reinterpret_cast<const float4*>(col + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                s[q] = v.x; s[q + 1] = v.y; s[q + 2] = v.z; s[q + 3] = v.w;
            }
            return;
        }
    }
#pragma unroll
    for (int q = 0; q < R; q++) {
        const int i = cd_channel<R>(lane, q);
        s[q] = ok && i < D ? col[i] : 0.0f;
    }
}
template <int R> __device__ __forceinline__ void cd_store_column(float* col, int lane, int D, bool ok, const float* s) {
    if (!ok) return;
    if constexpr (R >= 4) {
        if (D % 4 == 0) {
#pragma unroll
            for (int q = 0; q < R; q += 4) {
                const int i = cd_channel<R>(lane, q);
                if (i < D) *reinterpret_cast<float4*>(col + i) = make_float4(s[q], s[q + 1], s[q + 2], s[q + 3]);
            }
            return;
        }
    }
#pragma unroll
    for (int q = 0; q < R; q++) {
        const int i = cd_channel<R>(lane, q);
        if (i < D) col[i] = s[q];
    }
}

// --------------------------------------------------------------------------------------- split
// Columns [at0, at0 + n0) of proj into out0 and [at1, at1 + n1) into out1 (n1 may be 0).
__global__ void __launch_bounds__(256)
cd_split_kernel(const float* proj, int stride, int at0, int n0, void* out0, int at1, int n1, void* out1, int two_terms, int rows) {
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(proj);
    const int n = n0 + n1;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < (size_t)rows * n; i += (size_t)gridDim.x * blockDim.x) {
        const size_t r = i / n;
        int c = (int)(i - r * n);
        const bool second = c >= n0;
        if (second) c -= n0;
        const float v = proj[r * stride + (second ? at1 : at0) + c];
        const int width = second ? n1 : n0;
        void* out = second ? out1 : out0;
        if (two_terms) {
            bf16* o = (bf16*)out + r * 2 * width;
            const bf16 hi = __float2bfloat16_rn(v);
            o[c] = hi;
            o[width + c] = __float2bfloat16_rn(v - __bfloat162float(hi));
        } else {
            ((float*)out)[r * width + c] = v;
        }
    }
}

// proj: [rows, stride] float; out_i: [rows, n_i] float, or [rows, 2 n_i] bf16 with `two_terms` (hi, then lo).
extern "C" int bc_delta_split(const float* proj, int stride, int at0, int n0, void* out0, int at1, int n1, void* out1, int two_terms, int rows,
                              cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && n0 > 0 && n1 >= 0 && at0 >= 0 && at0 + n0 <= stride && at1 >= 0 && at1 + n1 <= stride, "delta_split: bad sizes");
    if (rows == 0) return BC_OK;
    const long long blocks = ((long long)rows * (n0 + n1) + 255) / 256;
    bc_launch(cd_split_kernel, dim3((unsigned)(blocks < 65535 ? blocks : 65535)), dim3(256), 0, s, proj, stride, at0, n0, out0, at1, n1, out1, two_terms, rows);
    BC_LAUNCH_STATUS();
}

// ------------------------------------------------------------------------------------- prepare
// qk: [rows, c_stride] float with q's G D values at 0 and k's at G D (changed in place to unit vectors, q over sqrt(D) too); z: [rows, H D]
// the decay's low-rank projection (changed in place to the decays); b: H numbers at proj + b_at; scal: [rows, H, 2] = (sigmoid(b), q . k).
__global__ void cd_prepare_kernel(float* qk, int c_stride, float* z, const float* proj, int stride, int b_at, const float* __restrict__ a_log,
                                  const float* __restrict__ dt_bias, float* __restrict__ scal, int rows, int H, int G, int D, float q_scale) {
    __shared__ float scratch[32];
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(qk); PDL_FRESH(z); PDL_FRESH(proj);
    const int row0 = blockIdx.x * CD_ROWS, h = blockIdx.y, rep = H / G, g = h / rep;
    const int n = min(CD_ROWS, rows - row0);
    const int d = threadIdx.x;
    const bool mine = d < D;
    const float a = -expf(a_log[h]), bias = mine ? dt_bias[h * D + d] : 0.0f;
    const bool owns = h % rep == 0;           // the first head of a group turns the shared q and k into unit vectors
    float* zc = z + (size_t)row0 * H * D + (size_t)h * D + d;
    float zv[CD_ROWS];
#pragma unroll
    for (int r = 0; r < CD_ROWS; r++) zv[r] = mine && r < n ? zc[(size_t)r * H * D] : 0.0f;
#pragma unroll
    for (int r = 0; r < CD_ROWS; r++)
        if (mine && r < n) zc[(size_t)r * H * D] = expf(a * cd_softplus(zv[r] + bias));
    if (d < n) scal[((size_t)(row0 + d) * H + h) * 2] = cd_sigmoid(proj[(size_t)(row0 + d) * stride + b_at + h]);
    if (!owns) return;
    float qv[CD_ROWS], kv[CD_ROWS];
#pragma unroll
    for (int r = 0; r < CD_ROWS; r++) {
        const float* p = qk + (size_t)(row0 + r) * c_stride + (size_t)g * D + d;
        qv[r] = mine && r < n ? p[0] : 0.0f;
        kv[r] = mine && r < n ? p[(size_t)G * D] : 0.0f;
    }
    for (int r = 0; r < n; r++) {
        float qr = 0.0f, kr = 0.0f;
#pragma unroll
        for (int i = 0; i < CD_ROWS; i++)
            if (i == r) qr = qv[i], kr = kv[i];
        const float qq = block_sum(qr * qr, scratch), kk = block_sum(kr * kr, scratch);
        const float q = qr / sqrtf(qq + CD_UNIT_EPS) * q_scale, k = kr / sqrtf(kk + CD_UNIT_EPS);
        const float dot = block_sum(q * k, scratch);
        if (mine) {
            float* p = qk + (size_t)(row0 + r) * c_stride + (size_t)g * D + d;
            p[0] = q;
            p[(size_t)G * D] = k;
        }
        if ((int)threadIdx.x < rep) scal[((size_t)(row0 + r) * H + h + threadIdx.x) * 2 + 1] = dot;
        for (int j = threadIdx.x + blockDim.x; j < rep; j += blockDim.x) scal[((size_t)(row0 + r) * H + h + j) * 2 + 1] = dot;
    }
}

extern "C" int bc_delta_channel_prepare(float* qk, int c_stride, float* z, const float* proj, int stride, int b_at, const float* a_log,
                                        const float* dt_bias, float* scal, int rows, int H, int G, int D, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && D > 0 && D <= CD_MAX_D, "delta_channel_prepare: bad sizes rows=%d H=%d G=%d D=%d",
                 rows, H, G, D);
    BC_CHECK_ARG(c_stride >= 2 * G * D && b_at >= 0 && b_at + H <= stride, "delta_channel_prepare: rows of %d and %d values do not hold q, k and b", c_stride, stride);
    if (rows == 0) return BC_OK;
    bc_launch(cd_prepare_kernel, dim3((rows + CD_ROWS - 1) / CD_ROWS, H), dim3((D + 31) / 32 * 32), 0, s, qk, c_stride, z, proj, stride, b_at, a_log, dt_bias,
              scal, rows, H, G, D, 1.0f / sqrtf((float)D));
    BC_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------------------- scan
__device__ __forceinline__ void cd_copy4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cd_copy16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cd_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cd_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <int R, int STEPS, bool VEC>      // key channels a thread (D <= 8 R), rows staged at a time, 16 bytes a copy
__global__ void __launch_bounds__(CD_LANES * CD_COLS)
cd_scan_kernel(const float* qkv, int c_stride, const float* decay, const float* scal, float* __restrict__ state, const int* __restrict__ seq_rows,
               const int* __restrict__ seq_slot, float* __restrict__ out, int H, int G, int D, int P, int n_slots, int write_state) {
    constexpr int DP = CD_LANES * R;
    constexpr int VECS = STEPS * DP;                               // one staged vector: [STEPS][DP]
    constexpr int BUF = 3 * VECS + STEPS * CD_BLOCK_COLS + STEPS * 2;
    __shared__ __align__(16) float sm[2][BUF];
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(qkv); PDL_FRESH(decay); PDL_FRESH(scal);
    const int sq = blockIdx.x, head = blockIdx.y, g = head / (H / G);
    const int slot = seq_slot[sq];
    const int row0 = seq_rows[sq], n_new = seq_rows[sq + 1] - row0;
    if (slot < 0 || slot >= n_slots || n_new <= 0) return;
    const int lane = threadIdx.x % CD_LANES, col = threadIdx.x / CD_LANES;
    const int jb = blockIdx.z * CD_BLOCK_COLS, j0 = jb + col;      // this thread's value channels: j0 and j0 + CD_COLS
    const int pv = min(CD_BLOCK_COLS, P - jb);
    // Channels past the head's width are never copied to: they stay zero.
    for (int e = threadIdx.x; e < 2 * BUF; e += blockDim.x) (&sm[0][0])[e] = 0.0f;
    __syncthreads();
    const float* qh = qkv + (size_t)g * D;
    const float* kh = qkv + (size_t)(G + g) * D;
    const float* vh = qkv + (size_t)2 * G * D + (size_t)head * P + jb;
    const float* dh = decay + (size_t)head * D;
    const size_t d_stride = (size_t)H * D;
    auto stage = [&](int t0, int b) {
        const int steps = min(STEPS, n_new - t0);
        float* base = sm[b];
        constexpr int W = VEC ? 4 : 1;
        const int nd = D / W, nv = pv / W;
        for (int e = threadIdx.x; e < steps * nd; e += blockDim.x) {
            const int t = e / nd, i = W * (e - t * nd);
            const size_t row = (size_t)(row0 + t0 + t);
            float* dst = base + t * DP + i;
            if (VEC) {
                cd_copy16(dst, dh + row * d_stride + i);
                cd_copy16(dst + VECS, qh + row * c_stride + i);
                cd_copy16(dst + 2 * VECS, kh + row * c_stride + i);
            } else {
                cd_copy4(dst, dh + row * d_stride + i);
                cd_copy4(dst + VECS, qh + row * c_stride + i);
                cd_copy4(dst + 2 * VECS, kh + row * c_stride + i);
            }
        }
        for (int e = threadIdx.x; e < steps * nv; e += blockDim.x) {
            const int t = e / nv, c = W * (e - t * nv);
            const float* src = vh + (size_t)(row0 + t0 + t) * c_stride + c;
            float* dst = base + 3 * VECS + t * CD_BLOCK_COLS + c;
            if (VEC) cd_copy16(dst, src);
            else cd_copy4(dst, src);
        }
        for (int e = threadIdx.x; e < steps * 2; e += blockDim.x)
            cd_copy4(base + 3 * VECS + STEPS * CD_BLOCK_COLS + e, scal + ((size_t)(row0 + t0 + e / 2) * H + head) * 2 + e % 2);
    };
    stage(0, 0);
    cd_commit();
    float* S = state + ((size_t)slot * H + head) * P * D;
    float s[CD_CJ][R];
    bool ok[CD_CJ];
#pragma unroll
    for (int cj = 0; cj < CD_CJ; cj++) {
        ok[cj] = j0 + cj * CD_COLS < P;
        cd_load_column<R>(S + (size_t)(ok[cj] ? j0 + cj * CD_COLS : 0) * D, lane, D, ok[cj], s[cj]);
    }
    int b = 0;
    for (int t0 = 0; t0 < n_new; t0 += STEPS, b ^= 1) {
        if (t0 + STEPS < n_new) stage(t0 + STEPS, b ^ 1);
        cd_commit();
        cd_wait<1>();
        __syncthreads();
        const int steps = min(STEPS, n_new - t0);
        const float *sw = sm[b], *sq_ = sw + VECS, *sk = sq_ + VECS, *sv = sk + VECS, *sd = sv + STEPS * CD_BLOCK_COLS;
        for (int t = 0; t < steps; t++) {
            float k[R], x[R], qw[CD_CJ], kw[CD_CJ];
            cd_load<R>(sw + t * DP, lane, x);
            cd_load<R>(sk + t * DP, lane, k);
#pragma unroll
            for (int cj = 0; cj < CD_CJ; cj++) {
                kw[cj] = 0.0f;
#pragma unroll
                for (int q = 0; q < R; q++) {
                    s[cj][q] *= x[q];
                    kw[cj] = fmaf(k[q], s[cj][q], kw[cj]);
                }
            }
            cd_load<R>(sq_ + t * DP, lane, x);
#pragma unroll
            for (int cj = 0; cj < CD_CJ; cj++) {
                qw[cj] = 0.0f;
#pragma unroll
                for (int q = 0; q < R; q++) qw[cj] = fmaf(x[q], s[cj][q], qw[cj]);
            }
#pragma unroll
            for (int o = CD_LANES / 2; o > 0; o >>= 1)
#pragma unroll
                for (int cj = 0; cj < CD_CJ; cj++) {
                    kw[cj] += __shfl_xor_sync(0xffffffffu, kw[cj], o);
                    qw[cj] += __shfl_xor_sync(0xffffffffu, qw[cj], o);
                }
            const float beta = sd[2 * t], qk = sd[2 * t + 1];
#pragma unroll
            for (int cj = 0; cj < CD_CJ; cj++) {
                const float r = beta * (sv[t * CD_BLOCK_COLS + cj * CD_COLS + col] - kw[cj]);
#pragma unroll
                for (int q = 0; q < R; q++) s[cj][q] = fmaf(k[q], r, s[cj][q]);
                if (lane == 0 && ok[cj]) out[((size_t)(row0 + t0 + t) * H + head) * P + j0 + cj * CD_COLS] = fmaf(qk, r, qw[cj]);
            }
        }
        __syncthreads();
    }
    cd_wait<0>();
    if (write_state) {
#pragma unroll
        for (int cj = 0; cj < CD_CJ; cj++) cd_store_column<R>(S + (size_t)(ok[cj] ? j0 + cj * CD_COLS : 0) * D, lane, D, ok[cj], s[cj]);
    }
}

// qkv: [rows, c_stride] float: q (G D), k (G D), v (H P); decay: [rows, H D]; scal: [rows, H, 2]; state: [n_slots, H, P, D] (value channel by
// value channel); out: [rows, H P].  Sequence s owns rows seq_rows[s] .. seq_rows[s + 1] and lives in slot seq_slot[s] (negative: skipped,
// its rows of `out` are left untouched).
extern "C" int bc_delta_channel_scan(const float* qkv, int c_stride, const float* decay, const float* scal, float* state, const int* seq_rows,
                                     const int* seq_slot, float* out, int seqs, int H, int G, int D, int P, int n_slots, int write_state,
                                     cudaStream_t s) {
    BC_CHECK_ARG(seqs >= 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && D > 0 && D <= CD_MAX_D && P > 0 && P <= 65535 * CD_BLOCK_COLS,
                 "delta_channel_scan: bad sizes seqs=%d H=%d G=%d D=%d P=%d (a head of at most %d)", seqs, H, G, D, P, CD_MAX_D);
    BC_CHECK_ARG(c_stride >= 2 * G * D + H * P, "delta_channel_scan: a row of %d values does not hold q, k and v", c_stride);
    if (seqs == 0) return BC_OK;
    const dim3 grid(seqs, H, (P + CD_BLOCK_COLS - 1) / CD_BLOCK_COLS), block(CD_LANES * CD_COLS);
    const bool vec = D % 4 == 0 && P % 4 == 0 && c_stride % 4 == 0 && (uintptr_t)qkv % 16 == 0 && (uintptr_t)decay % 16 == 0;
#define CD_CASE(R, STEPS)                                                                                                                               \
    do {                                                                                                                                                \
        if (vec) bc_launch(cd_scan_kernel<R, STEPS, true>, grid, block, 0, s, qkv, c_stride, decay, scal, state, seq_rows, seq_slot, out, H, G, D, P,   \
                           n_slots, write_state);                                                                                                      \
        else bc_launch(cd_scan_kernel<R, STEPS, false>, grid, block, 0, s, qkv, c_stride, decay, scal, state, seq_rows, seq_slot, out, H, G, D, P,      \
                       n_slots, write_state);                                                                                                          \
    } while (0)
    if (D <= 16) CD_CASE(2, 16);
    else if (D <= 32) CD_CASE(4, 16);
    else if (D <= 64) CD_CASE(8, 16);
    else if (D <= 128) CD_CASE(16, 8);
    else CD_CASE(32, 4);
#undef CD_CASE
    BC_LAUNCH_STATUS();
}

// ---------------------------------------------------------------------------------------- step
__device__ __forceinline__ float cd_dot_row(const float* w, const float* x, int n, int lane) {
    float a = 0.0f;
    for (int i = lane; i < n; i += 32) a = fmaf(w[i], x[i], a);
    return warp_sum(a);
}
__device__ __forceinline__ float cd_dot_row(const bf16* w, const float* x, int n, int lane) {
    float a = 0.0f;
    if (n % 4 == 0 && (uintptr_t)w % 8 == 0) {
        for (int i = 4 * lane; i < n; i += 128) {
            const uint2 raw = *reinterpret_cast<const uint2*>(w + i);
            const float4 v = *reinterpret_cast<const float4*>(x + i);
            a = fmaf(__uint_as_float(raw.x << 16), v.x, a); a = fmaf(__uint_as_float(raw.x & 0xffff0000u), v.y, a);
            a = fmaf(__uint_as_float(raw.y << 16), v.z, a); a = fmaf(__uint_as_float(raw.y & 0xffff0000u), v.w, a);
        }
    } else {
        for (int i = lane; i < n; i += 32) a = fmaf(to_f32(w[i]), x[i], a);
    }
    return warp_sum(a);
}

// Shared memory, in floats: inner vectors (each rounded up to 4), decay, q, k (DP each), v and the gate (P each), o (P).
template <int R, class T>
__global__ void __launch_bounds__(512)
cd_step_kernel(const float* qkv, int c_stride, const float* proj, int stride, int b_at, int a_at, int a_rank, int g_at, int g_rank, const T* __restrict__ wa2,
               const T* __restrict__ wg2, const float* __restrict__ a_log, const float* __restrict__ dt_bias, const float* __restrict__ norm_w,
               float* __restrict__ state, const int* __restrict__ row_slot, T* __restrict__ out, int H, int G, int D, int P, float q_scale, float eps,
               int n_slots, int write_state) {
    constexpr int DP = CD_LANES * R;
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    float* xa = sm;
    float* xg = xa + ((a_rank + 3) & ~3);
    float* sw = xg + ((g_rank + 3) & ~3);
    float *sq = sw + DP, *sk = sq + DP, *sg = sk + DP, *so = sg + P;
    pdl_launch_dependents_if_resident();
    pdl_wait();
    PDL_FRESH(qkv); PDL_FRESH(proj);
    const int row = blockIdx.x, head = blockIdx.y, g = head / (H / G);
    const int slot = row_slot[row];
    if (slot < 0 || slot >= n_slots) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const float* p = proj + (size_t)row * stride;
    const float* c = qkv + (size_t)row * c_stride;
    for (int i = threadIdx.x; i < a_rank; i += blockDim.x) xa[i] = p[a_at + i];
    for (int i = threadIdx.x; i < g_rank; i += blockDim.x) xg[i] = p[g_at + i];
    for (int i = threadIdx.x; i < 3 * DP; i += blockDim.x) sw[i] = 0.0f;
    __syncthreads();
    // The outer products, a warp an output: the head's D decays, then its P gates.
    const float a = -expf(a_log[head]);
#pragma unroll 4
    for (int i = warp; i < D + P; i += warps) {
        if (i < D) {
            const float z = cd_dot_row(wa2 + ((size_t)head * D + i) * a_rank, xa, a_rank, lane);
            if (lane == 0) sw[i] = expf(a * cd_softplus(z + dt_bias[head * D + i]));
        } else {
            const float z = cd_dot_row(wg2 + ((size_t)head * P + i - D) * g_rank, xg, g_rank, lane);
            if (lane == 0) sg[i - D] = cd_sigmoid(z);
        }
    }
    float qq = 0.0f, kk = 0.0f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        const float q = c[(size_t)g * D + d], k = c[(size_t)(G + g) * D + d];
        sq[d] = q;
        sk[d] = k;
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
    }
    qq = q_scale / sqrtf(block_sum(qq, scratch) + CD_UNIT_EPS);
    kk = 1.0f / sqrtf(block_sum(kk, scratch) + CD_UNIT_EPS);
    float dot = 0.0f;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        const float q = sq[d] * qq, k = sk[d] * kk;
        sq[d] = q;
        sk[d] = k;
        dot = fmaf(q, k, dot);
    }
    const float qk = block_sum(dot, scratch);             // its barriers also publish sq, sk, sw and sg
    const float beta = cd_sigmoid(p[b_at + head]);
    const int sub = threadIdx.x % CD_LANES;
    float w[R], k[R], q[R];
    cd_load<R>(sw, sub, w);
    cd_load<R>(sk, sub, k);
    cd_load<R>(sq, sub, q);
    float* S = state + ((size_t)slot * H + head) * P * D;
    const float* v = c + (size_t)2 * G * D + (size_t)head * P;
    const int per = blockDim.x / CD_LANES;
    for (int jb = 0; jb < P; jb += per) {                  // the same number of rounds for every thread: the shuffles need whole warps
        const int j = jb + (int)threadIdx.x / CD_LANES;
        const bool ok = j < P;
        float s[R], kw = 0.0f, qw = 0.0f;
        cd_load_column<R>(S + (size_t)(ok ? j : 0) * D, sub, D, ok, s);
        const float vj = ok ? v[j] : 0.0f;
#pragma unroll
        for (int i = 0; i < R; i++) {
            s[i] *= w[i];
            kw = fmaf(k[i], s[i], kw);
            qw = fmaf(q[i], s[i], qw);
        }
#pragma unroll
        for (int o = CD_LANES / 2; o > 0; o >>= 1) {
            kw += __shfl_xor_sync(0xffffffffu, kw, o);
            qw += __shfl_xor_sync(0xffffffffu, qw, o);
        }
        const float r = beta * (vj - kw);
        if (write_state) {
#pragma unroll
            for (int i = 0; i < R; i++) s[i] = fmaf(k[i], r, s[i]);
            cd_store_column<R>(S + (size_t)(ok ? j : 0) * D, sub, D, ok, s);
        }
        if (sub == 0 && ok) so[j] = fmaf(qk, r, qw);
    }
    __syncthreads();
    float ss = 0.0f;
    for (int j = threadIdx.x; j < P; j += blockDim.x) ss = fmaf(so[j], so[j], ss);
    const float f = 1.0f / sqrtf(block_sum(ss, scratch) / (float)P + eps);
    for (int j = threadIdx.x; j < P; j += blockDim.x) out[((size_t)row * H + head) * P + j] = from_f32<T>(so[j] * f * norm_w[j] * sg[j]);
}

template <class T>
static int step(const float* qkv, int c_stride, const float* proj, int stride, int b_at, int a_at, int a_rank, int g_at, int g_rank, const void* wa2,
                const void* wg2, const float* a_log, const float* dt_bias, const float* norm_w, float* state, const int* row_slot, void* out, int rows,
                int H, int G, int D, int P, float eps, int n_slots, int write_state, cudaStream_t s) {
    BC_CHECK_ARG(rows >= 0 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && D > 0 && D <= CD_MAX_D && P > 0 && P <= 2048,
                 "delta_channel_step: bad sizes rows=%d H=%d G=%d D=%d P=%d", rows, H, G, D, P);
    BC_CHECK_ARG(a_rank > 0 && g_rank > 0 && a_rank <= 2048 && g_rank <= 2048 && c_stride >= 2 * G * D + H * P, "delta_channel_step: bad ranks %d, %d or row of %d",
                 a_rank, g_rank, c_stride);
    if (rows == 0) return BC_OK;
    int threads = 64;
    while (threads < CD_LANES * P && threads < 512) threads *= 2;
    const dim3 grid(rows, H);
#define CD_STEP(R)                                                                                                                                        \
    bc_launch(cd_step_kernel<R, T>, grid, dim3(threads), (size_t)(((a_rank + 3) & ~3) + ((g_rank + 3) & ~3) + 3 * CD_LANES * R + 2 * P) * sizeof(float), s, \
              qkv, c_stride, proj, stride, b_at, a_at, a_rank, g_at, g_rank, (const T*)wa2, (const T*)wg2, a_log, dt_bias, norm_w, state, row_slot, (T*)out,  \
              H, G, D, P, 1.0f / sqrtf((float)D), eps, n_slots, write_state)
    if (D <= 16) CD_STEP(2);
    else if (D <= 32) CD_STEP(4);
    else if (D <= 64) CD_STEP(8);
    else if (D <= 128) CD_STEP(16);
    else CD_STEP(32);
#undef CD_STEP
    BC_LAUNCH_STATUS();
}

// One row a sequence (row r lives in slot row_slot[r]; negative: skipped, its row of `out` is left untouched).  qkv: [rows, c_stride], the
// convolved q, k (not yet unit vectors) and v; proj: [rows, stride] with b's H numbers at b_at and the inner vectors at a_at and g_at;
// wa2 [H D, a_rank], wg2 [H P, g_rank] and out [rows, H P] of the activation type.
extern "C" int bc_delta_channel_step_f32(const float* qkv, int c_stride, const float* proj, int stride, int b_at, int a_at, int a_rank, int g_at, int g_rank,
                                         const void* wa2, const void* wg2, const float* a_log, const float* dt_bias, const float* norm_w, float* state,
                                         const int* row_slot, void* out, int rows, int H, int G, int D, int P, float eps, int n_slots, int write_state,
                                         cudaStream_t s) {
    return step<float>(qkv, c_stride, proj, stride, b_at, a_at, a_rank, g_at, g_rank, wa2, wg2, a_log, dt_bias, norm_w, state, row_slot, out, rows, H, G, D, P,
                       eps, n_slots, write_state, s);
}
extern "C" int bc_delta_channel_step_bf16(const float* qkv, int c_stride, const float* proj, int stride, int b_at, int a_at, int a_rank, int g_at, int g_rank,
                                          const void* wa2, const void* wg2, const float* a_log, const float* dt_bias, const float* norm_w, float* state,
                                          const int* row_slot, void* out, int rows, int H, int G, int D, int P, float eps, int n_slots, int write_state,
                                          cudaStream_t s) {
    return step<bf16>(qkv, c_stride, proj, stride, b_at, a_at, a_rank, g_at, g_rank, wa2, wg2, a_log, dt_bias, norm_w, state, row_slot, out, rows, H, G, D, P,
                      eps, n_slots, write_state, s);
}
