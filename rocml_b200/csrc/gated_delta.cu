// The gated delta rule: a state per head that forgets by a decay and is corrected, token by token, towards v along k.
//
//   S <- g S;   w = beta (v - S^T k);   S <- S + k w^T;   o = S^T q          S [dim, vdim] per (sequence, head), 32-bit
//
// with g one number a head or one a key channel (a row of S).  With k and q the token's vectors and P = g S the decayed
// state, o = P^T q + w (k . q), so both sums over the rows are formed in one pass over the state and meet in one exchange.
//
//   delta_prep   everything between the projections and the recurrence: the short causal convolutions over time with
//                silu, q and k divided by their length (q times a constant as well), their dot product, the step size
//                beta = sigmoid(.), the decay g = exp(-exp(A) softplus(z + bias)); all 32-bit, into rows that the
//                recurrence copies straight to shared memory.  A block is (sequence, 32 tokens, unit), a unit the q and k
//                of one key head or one head's v, beta and g; a warp takes a token at a time.  What lies before a
//                sequence's first token of the step comes from its slot; the block of a sequence's first tokens
//                is the only one that reads the slot, and it leaves the step's last inputs there after its reads.
//   delta_scan   the recurrence.  A head's columns do not depend on one another: a warp owns four of them, sixteen lanes
//                each pair, and keeps its part of the state in registers from the step's first token to its last, so the
//                state is read and written once a step whatever the number of tokens.  A block has eight warps (or fewer, for
//                few columns); the tokens' q, k, g and v arrive in shared memory by cp.async, a batch of tokens ahead.
//                The order of a token's operations depends neither on how the prompt was cut nor on the batch.
//   delta_scan_chunks   the same for prompts, four tokens at a time: the sums over the rows of four tokens meet in one exchange.
//   low_rank     a narrow product through few inner values for few tokens (a decode step's W2 (W1 h)), 32-bit FMA.
#include "common.cuh"
#include "api.h"

using namespace rb;

namespace {
template <typename IT>
__device__ __forceinline__ float sum_in(const IT* p, int n_in, size_t in_stride) {
    float v = 0.f;
    for (int s = 0; s < n_in; s += 4) {                 // four partial sums in flight, added in order
        float y[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = s + j < n_in ? to_f32(p[(size_t)(s + j) * in_stride]) : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) v += y[j];
    }
    return v;
}
template <int VEC, typename IT>
__device__ __forceinline__ void sum_vec(const IT* p, int n_in, size_t in_stride, float* x) {
    if constexpr (VEC == 4) {
        x[0] = x[1] = x[2] = x[3] = 0.f;
        for (int s = 0; s < n_in; s += 4) {             // four partial sums in flight, added in order
            float y[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (s + j < n_in) load4(p + (size_t)(s + j) * in_stride, y[j]);
                else y[j][0] = y[j][1] = y[j][2] = y[j][3] = 0.f;
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int u = 0; u < 4; ++u) x[u] += y[j][u];
        }
    } else {
        x[0] = sum_in(p, n_in, in_stride);
    }
}
template <int VEC>
__device__ __forceinline__ void load_vec(const float* p, float* x) {
    if constexpr (VEC == 4) load4(p, x);
    else x[0] = p[0];
}
template <int VEC>
__device__ __forceinline__ void store_vec(float* p, const float* x) {
    if constexpr (VEC == 4) store4(p, x);
    else p[0] = x[0];
}
__device__ __forceinline__ float softplus_f32(float z) { return z > 20.f ? z : log1pf(expf(z)); }

constexpr int PREP_TOK = 32;          // tokens a block; more than a convolution's kept inputs
constexpr int PREP_MAX_TAPS = PREP_TOK;

struct PrepArgs {
    size_t in_stride;
    int n_in, row_stride, q_off, k_off, v_off, b_off;
    int heads, kv_heads, dim, vdim, taps, channels;
    const float* conv_w;              // [taps][channels]
    float* kept;                      // [slots][taps - 1][channels]
    size_t z_in_stride;
    int z_n_in, z_row_stride;
    const float *dt_bias, *a_log;
    int per_channel;
    float unit_eps, q_scale;
    const int *seq_slot, *cu_q;
    float* u;
    int ld_u, uq, uk, uv, ug, ub, ud;
};

// silu(convolution) of VEC neighbouring channels of token t: `col` their column in the projection rows, `c` their place among
// the convolution's channels.
template <int VEC, typename IT>
__device__ __forceinline__ void conv_silu(const PrepArgs& a, const IT* in, const float* mine, int t, int t_begin, int col, int c,
                                          float* acc) {
#pragma unroll
    for (int u = 0; u < VEC; ++u) acc[u] = 0.f;
    const int back = a.taps - 1;
    for (int j = 0; j < a.taps; ++j) {
        const int r = t - back + j;
        float x[VEC], w[VEC];
        if (r >= t_begin) sum_vec<VEC>(in + (size_t)r * a.row_stride + col, a.n_in, a.in_stride, x);
        else load_vec<VEC>(mine + (size_t)(back + (r - t_begin)) * a.channels + c, x);
        load_vec<VEC>(a.conv_w + (size_t)j * a.channels + c, w);
#pragma unroll
        for (int u = 0; u < VEC; ++u) acc[u] = fmaf(w[u], x[u], acc[u]);
    }
#pragma unroll
    for (int u = 0; u < VEC; ++u) acc[u] = silu(acc[u]);
}

// The slot's new rows for channels [c0, c0 + n): the last taps - 1 of (old rows, the step's rows).  A channel is one thread's,
// which reads every row before it overwrites it (a row comes from the same or a later place).
template <int VEC, typename IT>
__device__ __forceinline__ void keep_inputs(const PrepArgs& a, const IT* in, float* mine, int t_begin, int len, int col0, int c0,
                                            int n) {
    const int back = a.taps - 1;
    for (int i = threadIdx.x * VEC; i < n; i += blockDim.x * VEC)
        for (int j0 = 0; j0 < back; j0 += 4) {          // four rows in flight; a later group's rows are not written before they are read
            float x[4][VEC];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int at = len + j0 + j;
                if (j0 + j >= back) continue;
                if (at < back) load_vec<VEC>(mine + (size_t)at * a.channels + c0 + i, x[j]);
                else sum_vec<VEC>(in + (size_t)(t_begin + at - back) * a.row_stride + col0 + i, a.n_in, a.in_stride, x[j]);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (j0 + j < back) store_vec<VEC>(mine + (size_t)(j0 + j) * a.channels + c0 + i, x[j]);
        }
}

template <typename IT, typename ZT, int VEC>
__global__ void __launch_bounds__(128)
delta_prep_kernel(const IT* __restrict__ in, const ZT* __restrict__ z, const PrepArgs a) {
    // (no early signal to the kernel after this one: the recurrence's few blocks, placed while thousands of these wait for
    // their predecessor, would crowd on the multiprocessors with room left; decode steps gain from it)
    if (blockDim.x == 32) pdl_trigger();
    pdl_wait();
    const int b = blockIdx.z, slot = a.seq_slot[b];
    if (slot < 0) return;
    const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
    const int t0 = t_begin + blockIdx.y * PREP_TOK;
    if (t0 >= t_end) return;
    const int n = min(PREP_TOK, t_end - t0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    float* mine = a.taps > 1 ? a.kept + (size_t)slot * (a.taps - 1) * a.channels : nullptr;
    const int kd = a.kv_heads * a.dim;
    if ((int)blockIdx.x < a.kv_heads) {
        const int h = blockIdx.x, c = h * a.dim;
        for (int tt = warp; tt < n; tt += warps) {
            const int t = t0 + tt;
            float* uq = a.u + (size_t)t * a.ld_u + a.uq + c;
            float* uk = a.u + (size_t)t * a.ld_u + a.uk + c;
            float qq = 0.f, kk = 0.f, qk = 0.f;
            for (int i = lane * VEC; i < a.dim; i += 32 * VEC) {
                float q[VEC], k[VEC];
                conv_silu<VEC>(a, in, mine, t, t_begin, a.q_off + c + i, c + i, q);
                conv_silu<VEC>(a, in, mine, t, t_begin, a.k_off + c + i, kd + c + i, k);
#pragma unroll
                for (int u = 0; u < VEC; ++u) { qq = fmaf(q[u], q[u], qq); kk = fmaf(k[u], k[u], kk); qk = fmaf(q[u], k[u], qk); }
                store_vec<VEC>(uq + i, q);
                store_vec<VEC>(uk + i, k);
            }
            const float fq = a.q_scale / sqrtf(warp_sum(qq) + a.unit_eps), fk = 1.f / sqrtf(warp_sum(kk) + a.unit_eps);
            qk = warp_sum(qk);
            for (int i = lane * VEC; i < a.dim; i += 32 * VEC) {      // each lane its own values
                float q[VEC], k[VEC];
                load_vec<VEC>(uq + i, q);
                load_vec<VEC>(uk + i, k);
#pragma unroll
                for (int u = 0; u < VEC; ++u) { q[u] *= fq; k[u] *= fk; }
                store_vec<VEC>(uq + i, q);
                store_vec<VEC>(uk + i, k);
            }
            if (lane == 0) a.u[(size_t)t * a.ld_u + a.ud + h] = qk * fq * fk;
        }
        if (blockIdx.y == 0 && a.taps > 1) {
            __syncthreads();
            keep_inputs<VEC>(a, in, mine, t_begin, t_end - t_begin, a.q_off + c, c, a.dim);
            keep_inputs<VEC>(a, in, mine, t_begin, t_end - t_begin, a.k_off + c, kd + c, a.dim);
        }
        return;
    }
    const int h = blockIdx.x - a.kv_heads, c = h * a.vdim;
    const float rate = expf(a.a_log[h]);
    for (int tt = warp; tt < n; tt += warps) {
        const int t = t0 + tt;
        float* row = a.u + (size_t)t * a.ld_u;
        for (int i = lane * VEC; i < a.vdim; i += 32 * VEC) {
            float v[VEC];
            conv_silu<VEC>(a, in, mine, t, t_begin, a.v_off + c + i, 2 * kd + c + i, v);
            store_vec<VEC>(row + a.uv + c + i, v);
        }
        if (a.per_channel) {
            for (int i = lane * VEC; i < a.dim; i += 32 * VEC) {
                float g[VEC], bias[VEC];
                sum_vec<VEC>(z + (size_t)t * a.z_row_stride + (size_t)h * a.dim + i, a.z_n_in, a.z_in_stride, g);
                load_vec<VEC>(a.dt_bias + (size_t)h * a.dim + i, bias);
#pragma unroll
                for (int u = 0; u < VEC; ++u) g[u] = expf(-rate * softplus_f32(g[u] + bias[u]));
                store_vec<VEC>(row + a.ug + (size_t)h * a.dim + i, g);
            }
        } else if (lane == 1) {
            row[a.ug + h] = expf(-rate * softplus_f32(sum_in(z + (size_t)t * a.z_row_stride + h, a.z_n_in, a.z_in_stride) + a.dt_bias[h]));
        }
        if (lane == 0) row[a.ub + h] = sigmoid_f32(sum_in(in + (size_t)t * a.row_stride + a.b_off + h, a.n_in, a.in_stride));
    }
    if (blockIdx.y == 0 && a.taps > 1) {
        __syncthreads();
        keep_inputs<VEC>(a, in, mine, t_begin, t_end - t_begin, a.v_off + c, 2 * kd + c, a.vdim);
    }
}

// The same for prompts with at most four taps and heads of at most 128 (a lane holds four channels): a warp takes eight tokens in a
// row, asks for all their rows at once and slides the convolution's window over them in registers.
constexpr int ROWS_W = PREP_TOK / 4;       // tokens a warp (four warps a block)

template <int TAPS, typename IT>
__device__ __forceinline__ void conv_rows(const PrepArgs& a, const IT* in, const float* mine, int t0, int n, int t_begin, int col, int c,
                                          float (&y)[ROWS_W][4]) {
    float x[ROWS_W + TAPS - 1][4], w[TAPS][4];
#pragma unroll
    for (int i = 0; i < ROWS_W + TAPS - 1; ++i) {
        const int r = t0 - (TAPS - 1) + i;
        x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.f;
        if (i >= n + TAPS - 1) continue;
        if (r >= t_begin) load4(in + (size_t)r * a.row_stride + col, x[i]);
        else if (TAPS > 1) load4(mine + (size_t)(TAPS - 1 + (r - t_begin)) * a.channels + c, x[i]);
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load4(a.conv_w + (size_t)j * a.channels + c, w[j]);
#pragma unroll
    for (int i = 0; i < ROWS_W; ++i)
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            float acc = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j][u], x[i + j][u], acc);
            y[i][u] = silu(acc);
        }
}

template <typename IT, typename ZT, int TAPS>
__global__ void __launch_bounds__(128)
delta_prep_rows_kernel(const IT* __restrict__ in, const ZT* __restrict__ z, const PrepArgs a) {
    pdl_wait();                        // no early signal: see delta_prep_kernel
    const int b = blockIdx.z, slot = a.seq_slot[b];
    if (slot < 0) return;
    const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
    const int tb = t_begin + blockIdx.y * PREP_TOK;
    if (tb >= t_end) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = tb + warp * ROWS_W, n = min(ROWS_W, t_end - t0);
    float* mine = TAPS > 1 ? a.kept + (size_t)slot * (TAPS - 1) * a.channels : nullptr;
    const int kd = a.kv_heads * a.dim, i0 = lane * 4;
    const bool keys = (int)blockIdx.x < a.kv_heads;
    const int h = keys ? blockIdx.x : blockIdx.x - a.kv_heads;
    if (n > 0 && keys) {
        const int c = h * a.dim + i0;
        const bool on = i0 < a.dim;
        float q[ROWS_W][4] = {}, k[ROWS_W][4] = {};
        if (on) {
            conv_rows<TAPS>(a, in, mine, t0, n, t_begin, a.q_off + c, c, q);
            conv_rows<TAPS>(a, in, mine, t0, n, t_begin, a.k_off + c, kd + c, k);
        }
#pragma unroll
        for (int t = 0; t < ROWS_W; ++t) {
            float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
            for (int u = 0; u < 4; ++u) { qq = fmaf(q[t][u], q[t][u], qq); kk = fmaf(k[t][u], k[t][u], kk); qk = fmaf(q[t][u], k[t][u], qk); }
            const float fq = a.q_scale / sqrtf(warp_sum(qq) + a.unit_eps), fk = 1.f / sqrtf(warp_sum(kk) + a.unit_eps);
            qk = warp_sum(qk);
            if (t >= n) continue;
            float* row = a.u + (size_t)(t0 + t) * a.ld_u;
            if (on) {
#pragma unroll
                for (int u = 0; u < 4; ++u) { q[t][u] *= fq; k[t][u] *= fk; }
                store4(row + a.uq + c, q[t]);
                store4(row + a.uk + c, k[t]);
            }
            if (lane == 0) row[a.ud + h] = qk * fq * fk;
        }
    } else if (n > 0) {
        const float rate = expf(a.a_log[h]);
        if (i0 < a.vdim) {
            const int c = h * a.vdim + i0;
            float v[ROWS_W][4];
            conv_rows<TAPS>(a, in, mine, t0, n, t_begin, a.v_off + c, 2 * kd + c, v);
#pragma unroll
            for (int t = 0; t < ROWS_W; ++t)
                if (t < n) store4(a.u + (size_t)(t0 + t) * a.ld_u + a.uv + c, v[t]);
        }
        if (a.per_channel) {
            if (i0 < a.dim) {
                float g[ROWS_W][4], bias[4];
#pragma unroll
                for (int t = 0; t < ROWS_W; ++t)
                    if (t < n) load4(z + (size_t)(t0 + t) * a.z_row_stride + (size_t)h * a.dim + i0, g[t]);
                load4(a.dt_bias + (size_t)h * a.dim + i0, bias);
#pragma unroll
                for (int t = 0; t < ROWS_W; ++t) {
                    if (t >= n) continue;
#pragma unroll
                    for (int u = 0; u < 4; ++u) g[t][u] = expf(-rate * softplus_f32(g[t][u] + bias[u]));
                    store4(a.u + (size_t)(t0 + t) * a.ld_u + a.ug + (size_t)h * a.dim + i0, g[t]);
                }
            }
        } else if (lane >= 16 && lane - 16 < n) {
            const int t = t0 + lane - 16;
            a.u[(size_t)t * a.ld_u + a.ug + h] = expf(-rate * softplus_f32(to_f32(z[(size_t)t * a.z_row_stride + h]) + a.dt_bias[h]));
        }
        if (lane < n) {
            const int t = t0 + lane;
            a.u[(size_t)t * a.ld_u + a.ub + h] = sigmoid_f32(to_f32(in[(size_t)t * a.row_stride + a.b_off + h]));
        }
    }
    if (blockIdx.y == 0 && TAPS > 1) {
        __syncthreads();
        if (keys) {
            keep_inputs<4>(a, in, mine, t_begin, t_end - t_begin, a.q_off + h * a.dim, h * a.dim, a.dim);
            keep_inputs<4>(a, in, mine, t_begin, t_end - t_begin, a.k_off + h * a.dim, kd + h * a.dim, a.dim);
        } else {
            keep_inputs<4>(a, in, mine, t_begin, t_end - t_begin, a.v_off + h * a.vdim, 2 * kd + h * a.vdim, a.vdim);
        }
    }
}

// ---- the recurrence ---------------------------------------------------------------------------------------------
constexpr int RL = 16;                // lanes that share a column's rows
constexpr int WCOLS = 4;              // columns a warp owns: two for each half of the warp

struct ScanArgs {
    const float* u;
    int ld_u, uq, uk, uv, ug, ub, ud;
    int heads, kv_heads, dim, vdim;
    float* state;                     // [slots][heads][vdim][dim]
    const int *seq_slot, *cu_q;
    float* out;
    int ld_out;
    int vec;                          // rows and pieces of them start on 16 bytes
};

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// R4: groups of four rows a lane holds (dim <= 64 R4).  CH: a decay per key channel.  TB: tokens staged at a time.
template <int R4, bool CH, int TB>
__global__ void __launch_bounds__(256)
delta_scan_kernel(const ScanArgs a) {
    pdl_trigger();
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = 64 * R4;                         // rows of a staged vector, zeros beyond dim
    constexpr int NV = CH ? 3 : 2;                      // q, k (, g)
    const int warps = blockDim.x >> 5;
    const int cols = warps * WCOLS;
    const int tok = NV * DP + cols + 4;                 // a staged token: q | k (| g) | v of this block's columns | beta, q.k, g
    float* outs = sm + 2 * TB * tok;                    // [TB][cols]
    const int b = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * cols;
    const int slot = a.seq_slot[b];
    if (slot < 0) return;
    const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
    if (t_end <= t_begin) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane & 15, half = lane >> 4;
    const int kvh = h / (a.heads / a.kv_heads);
    const int jl = warp * WCOLS + half * 2;             // this lane's two columns: jl, jl + 1 of the block's

    // the state: written by an earlier step, so it is read before this step's kernels are waited for
    float S[2][R4][4];
    float* st = a.state + ((size_t)slot * a.heads + h) * a.vdim * a.dim;
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int j = j0 + jl + c;
#pragma unroll
        for (int r = 0; r < R4; ++r) {
            const int i = (r * RL + l) * 4;
            S[c][r][0] = S[c][r][1] = S[c][r][2] = S[c][r][3] = 0.f;
            if (j < a.vdim) {
                if ((a.dim & 3) == 0) {
                    if (i < a.dim) load4(st + (size_t)j * a.dim + i, S[c][r]);
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e) if (i + e < a.dim) S[c][r][e] = st[(size_t)j * a.dim + i + e];
                }
            }
        }
    }
    if (a.dim < DP || j0 + cols > a.vdim)               // what no copy fills stays zero
        for (int i = threadIdx.x; i < 2 * TB * tok; i += blockDim.x) sm[i] = 0.f;
    __syncthreads();
    pdl_wait();

    const int nv = min(cols, a.vdim - j0);
    auto stage = [&](int t0, int buf) {
        const int nb = min(TB, t_end - t0);
        float* base = sm + buf * TB * tok;
        const float* u0 = a.u + (size_t)t0 * a.ld_u;
        if (a.vec) {
            const int d4 = a.dim >> 2, v4 = nv >> 2, per = NV * d4 + v4;
            for (int i = threadIdx.x; i < nb * per; i += blockDim.x) {
                const int tt = i / per;
                int x = i - tt * per;
                const float* row = u0 + (size_t)tt * a.ld_u;
                float* dst = base + tt * tok;
                if (x < d4) cp_async16(dst + 4 * x, row + a.uq + kvh * a.dim + 4 * x);
                else if ((x -= d4) < d4) cp_async16(dst + DP + 4 * x, row + a.uk + kvh * a.dim + 4 * x);
                else if (CH && (x -= d4) < d4) cp_async16(dst + 2 * DP + 4 * x, row + a.ug + (size_t)h * a.dim + 4 * x);
                else {
                    cp_async16(dst + NV * DP + 4 * (x - d4), row + a.uv + (size_t)h * a.vdim + j0 + 4 * (x - d4));
                }
            }
        } else {
            const int per = NV * a.dim + nv;
            for (int i = threadIdx.x; i < nb * per; i += blockDim.x) {
                const int tt = i / per, x = i - tt * per;
                const float* row = u0 + (size_t)tt * a.ld_u;
                float* dst = base + tt * tok;
                const int what = x / a.dim, e = x - what * a.dim;
                if (what == 0) cp_async4(dst + e, row + a.uq + kvh * a.dim + e);
                else if (what == 1) cp_async4(dst + DP + e, row + a.uk + kvh * a.dim + e);
                else if (CH && what == 2) cp_async4(dst + 2 * DP + e, row + a.ug + (size_t)h * a.dim + e);
                else cp_async4(dst + NV * DP + (x - NV * a.dim), row + a.uv + (size_t)h * a.vdim + j0 + (x - NV * a.dim));
            }
        }
        for (int i = threadIdx.x; i < nb; i += blockDim.x) {
            const float* row = u0 + (size_t)i * a.ld_u;
            float* dst = base + i * tok + NV * DP + cols;
            cp_async4(dst, row + a.ub + h);
            cp_async4(dst + 1, row + a.ud + kvh);
            if (!CH) cp_async4(dst + 2, row + a.ug + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    stage(t_begin, 0);
    int buf = 0;
    for (int t0 = t_begin; t0 < t_end; t0 += TB, buf ^= 1) {
        const int nb = min(TB, t_end - t0);
        if (t0 + TB < t_end) {
            stage(t0 + TB, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float* base = sm + buf * TB * tok;
        for (int tt = 0; tt < nb; ++tt) {
            const float* x = base + tt * tok;
            const float* sc = x + NV * DP + cols;
            const float beta = sc[0], dot = sc[1];
            const float gh = CH ? 0.f : sc[2];
            const float v0 = x[NV * DP + jl], v1 = x[NV * DP + jl + 1];
            float k[R4][4];
            float ak0 = 0.f, ak1 = 0.f, aq0 = 0.f, aq1 = 0.f;
#pragma unroll
            for (int r = 0; r < R4; ++r) {
                const int i = (r * RL + l) * 4;
                float q[4], g[4];
                load4(x + i, q);
                load4(x + DP + i, k[r]);
                if (CH) load4(x + 2 * DP + i, g);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float f = CH ? g[e] : gh;
                    const float s0 = f * S[0][r][e], s1 = f * S[1][r][e];
                    S[0][r][e] = s0;
                    S[1][r][e] = s1;
                    ak0 = fmaf(k[r][e], s0, ak0);
                    ak1 = fmaf(k[r][e], s1, ak1);
                    aq0 = fmaf(q[e], s0, aq0);
                    aq1 = fmaf(q[e], s1, aq1);
                }
            }
            // four sums over sixteen lanes: halves exchange what the other keeps; lanes 0-3 end with k . column 0, 4-7 with
            // k . column 1, 8-11 and 12-15 with q's
            const bool up8 = (lane & 8) != 0, up4 = (lane & 4) != 0;
            float x0 = up8 ? aq0 : ak0, x1 = up8 ? aq1 : ak1;
            x0 += __shfl_xor_sync(0xffffffffu, up8 ? ak0 : aq0, 8);
            x1 += __shfl_xor_sync(0xffffffffu, up8 ? ak1 : aq1, 8);
            float y = up4 ? x1 : x0;
            y += __shfl_xor_sync(0xffffffffu, up4 ? x0 : x1, 4);
            y += __shfl_xor_sync(0xffffffffu, y, 2);
            y += __shfl_xor_sync(0xffffffffu, y, 1);
            const float w0 = beta * (v0 - __shfl_sync(0xffffffffu, y, lane & 16));
            const float w1 = beta * (v1 - __shfl_sync(0xffffffffu, y, (lane & 16) | 4));
            if (l == 8) outs[tt * cols + jl] = fmaf(w0, dot, y);
            if (l == 12) outs[tt * cols + jl + 1] = fmaf(w1, dot, y);
#pragma unroll
            for (int r = 0; r < R4; ++r)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    S[0][r][e] = fmaf(k[r][e], w0, S[0][r][e]);
                    S[1][r][e] = fmaf(k[r][e], w1, S[1][r][e]);
                }
        }
        __syncthreads();                                // the results are there, and the buffer may be filled again
        for (int i = threadIdx.x; i < nb * cols; i += blockDim.x) {
            const int tt = i / cols, j = i - tt * cols;
            if (j < nv) a.out[(size_t)(t0 + tt) * a.ld_out + (size_t)h * a.vdim + j0 + j] = outs[i];
        }
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
        const int j = j0 + jl + c;
        if (j >= a.vdim) continue;
#pragma unroll
        for (int r = 0; r < R4; ++r) {
            const int i = (r * RL + l) * 4;
            if ((a.dim & 3) == 0) {
                if (i < a.dim) store4(st + (size_t)j * a.dim + i, S[c][r]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) if (i + e < a.dim) st[(size_t)j * a.dim + i + e] = S[c][r][e];
            }
        }
    }
}

// Warps a block: few (columns) while the grid would not fill the device otherwise, eight beyond.
int scan_warps(int n_seqs, int n_heads, int vdim) {
    int warps = 8;
    const long long heads = (long long)n_seqs * n_heads;
    while (warps > 1 && (heads * ((vdim + warps * WCOLS - 1) / (warps * WCOLS)) < 148 || (warps - 1) * WCOLS >= vdim)) warps >>= 1;
    return warps < 4 && vdim > 2 * WCOLS ? 4 : warps;
}

template <int R4, bool CH, int TB>
int launch_scan(const ScanArgs& a, int n_seqs, cudaStream_t s) {
    const int warps = scan_warps(n_seqs, a.heads, a.vdim), cols = warps * WCOLS;
    const size_t smem = ((size_t)2 * TB * ((CH ? 3 : 2) * 64 * R4 + cols + 4) + (size_t)TB * cols) * sizeof(float);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    auto k = delta_scan_kernel<R4, CH, TB>;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    RB_LAUNCH((k), dim3((a.vdim + cols - 1) / cols, a.heads, n_seqs), dim3(warps * 32), smem, s, a);
    RB_LAUNCH_CHECK();
    return RB_OK;
}

// ---- prompts: four tokens at a time -------------------------------------------------------------------------------
// With S the state before a chunk of four tokens, G_t = g_1 .. g_t the decays up to token t inside it and G_(t,s) = g_(s+1) .. g_t:
//   a_t = (G_t k_t)^T S + sum_{s < t} (k_t . G_(t,s) k_s) w_s,   w_t = beta_t (v_t - a_t)
//   o_t = (G_t q_t)^T S + sum_{s <= t} (q_t . G_(t,s) k_s) w_s,   S' = G_4 S + sum_s (G_(4,s) k_s) w_s^T
// so the columns' lanes exchange their sums once for four tokens instead of once a token, and no decay multiplies the state
// but the chunk's.  Every G is a product of decays (no quotient), so nothing overflows.  delta_chunk forms the vectors G_t q_t,
// G_t k_t, G_(4,s) k_s, the decay G_4 and the two triangles of products, once for all columns.
constexpr int CH_T = 4;
constexpr int CH_SCAL = 36;            // a chunk's numbers: [4][4] of k . k, [4][4] of q . k, four step sizes

// One warp a (chunk, head).  vecs [heads][T][3][dimp]; firsts [heads][n_chunks][dimp + 36], a chunk's decay and numbers.  The
// chunks of sequence b are numbered from cu_q[b] / 4 + b, so that no two sequences share a number.
__global__ void __launch_bounds__(128)
delta_chunk_kernel(const float* __restrict__ u, int ld_u, int uq, int uk, int ug, int ub, int heads, int kv_heads, int dim, int dimp,
                   int per_channel, const int* __restrict__ seq_slot, const int* __restrict__ cu_q, int T, int n_chunks,
                   float* __restrict__ vecs, float* __restrict__ firsts) {
    pdl_wait();                        // no early signal: see delta_prep_kernel
    const int b = blockIdx.z;
    if (seq_slot[b] < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = cu_q[b] + (blockIdx.x * 4 + warp) * CH_T, t_end = cu_q[b + 1];
    if (t0 >= t_end) return;
    const int n = min(CH_T, t_end - t0), h = blockIdx.y, kvh = h / (heads / kv_heads);
    const int chunk = cu_q[b] / CH_T + b + blockIdx.x * 4 + warp;
    float* first = firsts + ((size_t)h * n_chunks + chunk) * (dimp + CH_SCAL);
    float kk[16], qk[16];              // [t][s], s <= t used
#pragma unroll
    for (int i = 0; i < 16; ++i) kk[i] = qk[i] = 0.f;
    for (int i = lane; i < dimp; i += 32) {
        float g[4], k[4], q[4];
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            const float* row = u + (size_t)(t0 + t) * ld_u;
            const bool in = t < n && i < dim;
            q[t] = in ? row[uq + kvh * dim + i] : 0.f;
            k[t] = in ? row[uk + kvh * dim + i] : 0.f;
            g[t] = in ? row[ug + (per_channel ? h * dim + i : h)] : 1.f;
        }
        float up = 1.f;                // G_t
        float part[4];                 // G_(t,s) k_s as t grows
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            up *= g[t];
#pragma unroll
            for (int s = 0; s < t; ++s) part[s] *= g[t];
            part[t] = k[t];
#pragma unroll
            for (int s = 0; s <= t; ++s) {
                kk[t * 4 + s] = fmaf(k[t], part[s], kk[t * 4 + s]);
                qk[t * 4 + s] = fmaf(q[t], part[s], qk[t * 4 + s]);
            }
            if (t < n) {
                float* dst = vecs + ((size_t)h * T + t0 + t) * 3 * dimp + i;
                dst[0] = up * q[t];
                dst[dimp] = up * k[t];
            }
        }
#pragma unroll
        for (int t = 0; t < 4; ++t)
            if (t < n) vecs[((size_t)h * T + t0 + t) * 3 * dimp + 2 * dimp + i] = part[t];
        first[i] = up;
    }
    // thirty-two sums over thirty-two lanes, each lane ending with one: kk 0..15, qk 16..31
    float x[32];
#pragma unroll
    for (int i = 0; i < 16; ++i) { x[i] = kk[i]; x[16 + i] = qk[i]; }
#pragma unroll
    for (int m = 16; m >= 1; m >>= 1) {
        const bool upper = (lane & m) != 0;
#pragma unroll
        for (int i = 0; i < m; ++i) {
            const float send = upper ? x[i] : x[i + m], keep = upper ? x[i + m] : x[i];
            x[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
        }
    }
    float* num = first + dimp;
    const int t = (lane >> 2) & 3, s = lane & 3;
    num[lane] = lane < 16 ? (s < t ? x[0] : 0.f) : (s <= t ? x[0] : 0.f);
    if (lane < 4) num[32 + lane] = lane < n ? u[(size_t)(t0 + lane) * ld_u + ub + h] : 0.f;
}

struct ChunkArgs {
    const float *u, *vecs, *firsts;
    int T, n_chunks, ld_u, uv, heads, dim, vdim, dimp;
    float* state;                     // [slots][heads][vdim][dim]
    const int *seq_slot, *cu_q;
    float* out;
    int ld_out, vec;                  // vec: v's columns start on 16 bytes
};

// Two 32-bit numbers a register pair: one instruction for two multiply-adds.
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ void unpack2(uint64_t v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ void load22(const float* p, uint64_t* x) {
    const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
    x[0] = v.x;
    x[1] = v.y;
}

// The recurrence over chunks: lanes and columns as in delta_scan_kernel (R4: groups of four rows a lane holds, dimp = 64 R4),
// four warps of columns a block, and a fifth warp that brings the next TB tokens and takes the last ones' results away, so
// that the warps of columns meet it once for TB tokens and do nothing else.
constexpr int CH_WARPS = 4;

template <int R4, int TB>
__global__ void __launch_bounds__((CH_WARPS + 1) * 32, R4 > 2 ? 1 : (TB <= 8 ? 4 : 3))
delta_scan_chunks_kernel(const ChunkArgs a) {
    extern __shared__ __align__(16) float sm[];
    constexpr int DP = 64 * R4, NCH = TB / CH_T, cols = CH_WARPS * WCOLS;
    constexpr int TOK = 3 * DP, CHK = DP + CH_SCAL;                 // a staged token's vectors; a staged chunk's decay and numbers
    constexpr int BUF = TB * (TOK + cols) + NCH * CHK;              // [TB][TOK] | [NCH][CHK] | [TB][cols] (v)
    float* outs = sm + 2 * BUF;                                     // [2][TB][cols]
    const int b = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * cols;
    const int slot = a.seq_slot[b];
    if (slot < 0) return;
    const int t_begin = a.cu_q[b], t_end = a.cu_q[b + 1];
    if (t_end <= t_begin) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l = lane & 15, half = lane >> 4;
    const int jl = (warp & (CH_WARPS - 1)) * WCOLS + half * 2;
    const int nv = min(cols, a.vdim - j0);
    const int batches = (t_end - t_begin + TB - 1) / TB;
    float* st = a.state + ((size_t)slot * a.heads + h) * a.vdim * a.dim;
    for (int i = threadIdx.x; i < 2 * BUF; i += blockDim.x) sm[i] = 0.f;            // columns beyond vdim stay zero
    __syncthreads();
    pdl_wait();

    if (warp == CH_WARPS) {
        auto stage = [&](int it) {
            const int t0 = t_begin + it * TB, nb = min(TB, t_end - t0), nc = (nb + CH_T - 1) / CH_T;
            float* base = sm + (it & 1) * BUF;
            const float* vec = a.vecs + ((size_t)h * a.T + t0) * TOK;
            for (int i = lane; i < nb * (TOK / 4); i += 32) cp_async16(base + 4 * i, vec + 4 * i);
            const float* fst = a.firsts + ((size_t)h * a.n_chunks + t_begin / CH_T + b + it * NCH) * CHK;
            for (int i = lane; i < nc * (CHK / 4); i += 32) cp_async16(base + TB * TOK + 4 * i, fst + 4 * i);
            float* vs = base + TB * TOK + NCH * CHK;
            const float* src = a.u + (size_t)t0 * a.ld_u + a.uv + (size_t)h * a.vdim + j0;
            if (a.vec) {
                for (int i = lane; i < nb * (cols / 4); i += 32) {
                    const int tt = i / (cols / 4), x = 4 * (i % (cols / 4));
                    if (x < nv) cp_async16(vs + tt * cols + x, src + (size_t)tt * a.ld_u + x);
                }
            } else {
                for (int i = lane; i < nb * cols; i += 32) {
                    const int tt = i / cols, x = i % cols;
                    if (x < nv) cp_async4(vs + tt * cols + x, src + (size_t)tt * a.ld_u + x);
                }
            }
            // a last chunk's missing tokens: nothing is added, nothing read
            for (int i = nb * TOK + lane; i < nc * CH_T * TOK; i += 32) base[i] = 0.f;
            for (int i = nb * cols + lane; i < nc * CH_T * cols; i += 32) vs[i] = 0.f;
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        auto take = [&](int it) {
            const int t0 = t_begin + it * TB, nb = min(TB, t_end - t0);
            const float* src = outs + (it & 1) * TB * cols;
            float* dst = a.out + (size_t)t0 * a.ld_out + (size_t)h * a.vdim + j0;
            for (int i = lane; i < nb * cols; i += 32) {
                const int tt = i / cols, x = i % cols;
                if (x < nv) dst[(size_t)tt * a.ld_out + x] = src[i];
            }
        };
        stage(0);
        for (int it = 0; it < batches; ++it) {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
            __syncthreads();                            // batch `it` is there; the warps of columns are done with the one before
            if (it + 1 < batches) stage(it + 1);
            if (it > 0) take(it - 1);
        }
        __syncthreads();
        take(batches - 1);
        return;
    }

    uint64_t S[2][R4][2];                               // rows in pairs
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int r = 0; r < R4; ++r) {
            float x[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = (r * RL + l) * 4 + e, j = j0 + jl + c;
                x[e] = i < a.dim && j < a.vdim ? st[(size_t)j * a.dim + i] : 0.f;
            }
            S[c][r][0] = pack2(x[0], x[1]);
            S[c][r][1] = pack2(x[2], x[3]);
        }
    for (int it = 0; it < batches; ++it) {
        const int nc = (min(TB, t_end - t_begin - it * TB) + CH_T - 1) / CH_T;
        const float* base = sm + (it & 1) * BUF;
        const float* vs = base + TB * TOK + NCH * CHK;
        float* res = outs + (it & 1) * TB * cols;
        __syncthreads();
        for (int cc = 0; cc < nc; ++cc) {
            const float* x = base + cc * CH_T * TOK;
            const float* dec = base + TB * TOK + cc * CHK;
            const float* num = dec + DP;
            float y[16];                 // [k | q][column][token]
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                uint64_t yk0 = 0, yk1 = 0, yq0 = 0, yq1 = 0;
#pragma unroll
                for (int r = 0; r < R4; ++r) {
                    uint64_t q[2], k[2];
                    load22(x + t * TOK + (r * RL + l) * 4, q);
                    load22(x + t * TOK + DP + (r * RL + l) * 4, k);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        yk0 = fma2(k[e], S[0][r][e], yk0);
                        yk1 = fma2(k[e], S[1][r][e], yk1);
                        yq0 = fma2(q[e], S[0][r][e], yq0);
                        yq1 = fma2(q[e], S[1][r][e], yq1);
                    }
                }
                float lo, hi;
                unpack2(yk0, lo, hi); y[t] = lo + hi;
                unpack2(yk1, lo, hi); y[4 + t] = lo + hi;
                unpack2(yq0, lo, hi); y[8 + t] = lo + hi;
                unpack2(yq1, lo, hi); y[12 + t] = lo + hi;
            }
            // what the corrections need is asked for before the sums are exchanged
            float tri[4][4], beta[4], v[2][4], d[4];
            load4(num + 32, beta);
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                load4(num + 4 * t, tri[t]);
                const float2 vv = *reinterpret_cast<const float2*>(vs + (cc * CH_T + t) * cols + jl);
                v[0][t] = vv.x;
                v[1][t] = vv.y;
            }
            load4(num + 16 + (l & 3) * 4, d);
            // sixteen sums over sixteen lanes: lane l ends with the l-th
#pragma unroll
            for (int m = 8; m >= 1; m >>= 1) {
                const bool upper = (l & m) != 0;
#pragma unroll
                for (int i = 0; i < m; ++i) {
                    const float send = upper ? y[i] : y[i + m], keep = upper ? y[i + m] : y[i];
                    y[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                }
            }
            float w[2][4];
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int t = 0; t < 4; ++t) w[c][t] = __shfl_sync(0xffffffffu, y[0], (lane & 16) | (c * 4 + t));
#pragma unroll
            for (int r = 0; r < R4; ++r) {
                uint64_t f[2];
                load22(dec + (r * RL + l) * 4, f);
#pragma unroll
                for (int e = 0; e < 2; ++e) { S[0][r][e] = mul2(S[0][r][e], f[e]); S[1][r][e] = mul2(S[1][r][e], f[e]); }
            }
#pragma unroll
            for (int t = 0; t < 4; ++t)
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    float at = w[c][t];
#pragma unroll
                    for (int s = 0; s < t; ++s) at = fmaf(tri[t][s], w[c][s], at);
                    w[c][t] = beta[t] * (v[c][t] - at);
                }
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const uint64_t w0 = pack2(w[0][t], w[0][t]), w1 = pack2(w[1][t], w[1][t]);
#pragma unroll
                for (int r = 0; r < R4; ++r) {
                    uint64_t ks[2];
                    load22(x + t * TOK + 2 * DP + (r * RL + l) * 4, ks);
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        S[0][r][e] = fma2(ks[e], w0, S[0][r][e]);
                        S[1][r][e] = fma2(ks[e], w1, S[1][r][e]);
                    }
                }
            }
            if (l >= 8) {
                const int c = (l >> 2) & 1;
                float o = y[0];
#pragma unroll
                for (int s = 0; s < 4; ++s) o = fmaf(d[s], c ? w[1][s] : w[0][s], o);
                res[(cc * CH_T + (l & 3)) * cols + jl + c] = o;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int r = 0; r < R4; ++r) {
            float x[4];
            unpack2(S[c][r][0], x[0], x[1]);
            unpack2(S[c][r][1], x[2], x[3]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = (r * RL + l) * 4 + e, j = j0 + jl + c;
                if (i < a.dim && j < a.vdim) st[(size_t)j * a.dim + i] = x[e];
            }
        }
}

template <int R4, int TB>
int launch_chunks(const ChunkArgs& a, int n_seqs, cudaStream_t s) {
    const int cols = CH_WARPS * WCOLS;
    const size_t smem = ((size_t)2 * (TB * (3 * 64 * R4 + cols) + TB / CH_T * (64 * R4 + CH_SCAL)) + (size_t)2 * TB * cols) * sizeof(float);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    auto k = delta_scan_chunks_kernel<R4, TB>;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    RB_LAUNCH((k), dim3((a.vdim + cols - 1) / cols, a.heads, n_seqs), dim3((CH_WARPS + 1) * 32), smem, s, a);
    RB_LAUNCH_CHECK();
    return RB_OK;
}

// ---- W2 x for few tokens ------------------------------------------------------------------------------------------
constexpr int LR_TOK = 8;
struct LowRank {
    const void *w0, *w1;
    int x0, rank0, n0, x1, rank1, n1;
};

// A block takes 64 rows of one matrix for eight tokens, four lanes a row: a lane multiplies eight neighbouring weights in turn
// with the tokens' inner values (shared memory, eight tokens a value, laid out so that the four lanes meet no bank twice).
constexpr int LR_ROWS = 64;
__device__ __forceinline__ int lr_at(int r) { return (r >> 3) * 72 + (r & 7) * LR_TOK; }

template <typename IT, typename WT>
__global__ void __launch_bounds__(4 * LR_ROWS)
low_rank_kernel(const IT* __restrict__ in, int n_in, size_t in_stride, int row_stride, const LowRank p, int T,
                float* __restrict__ out, int ld_out) {
    pdl_trigger();
    extern __shared__ __align__(16) float xs[];        // [rank][LR_TOK], see lr_at
    const int blocks0 = (p.n0 + LR_ROWS - 1) / LR_ROWS;
    const bool second = (int)blockIdx.x >= blocks0;
    const int rank = second ? p.rank1 : p.rank0, n = second ? p.n1 : p.n0, x_off = second ? p.x1 : p.x0;
    const WT* w = static_cast<const WT*>(second ? p.w1 : p.w0);
    const int row = ((int)blockIdx.x - (second ? blocks0 : 0)) * LR_ROWS + (threadIdx.x >> 2), sub = threadIdx.x & 3;
    const int t0 = blockIdx.y * LR_TOK;
    const bool vec = (rank & 7) == 0 && ((uintptr_t)w & (4 * sizeof(WT) - 1)) == 0;
    const WT* wr = w + (size_t)(row < n ? row : 0) * rank;
    // the weights do not depend on the kernel before this one: a lane's first sixteen are asked for before the wait
    float first[2][8];
#pragma unroll
    for (int c = 0; c < 2; ++c)
        if (vec && (c * 4 + sub) * 8 < rank) { load4(wr + (c * 4 + sub) * 8, first[c]); load4(wr + (c * 4 + sub) * 8 + 4, first[c] + 4); }
    pdl_wait();
    for (int i = threadIdx.x; i < rank * LR_TOK; i += 4 * LR_ROWS) {
        const int tt = i / rank, r = i - tt * rank;
        xs[lr_at(r) + tt] = t0 + tt < T ? sum_in(in + (size_t)(t0 + tt) * row_stride + x_off + r, n_in, in_stride) : 0.f;
    }
    __syncthreads();
    float acc[LR_TOK] = {};
    auto add = [&](float wv, int r) {
        const float* x = xs + lr_at(r);
        const float4 lo = *reinterpret_cast<const float4*>(x), hi = *reinterpret_cast<const float4*>(x + 4);
        acc[0] = fmaf(wv, lo.x, acc[0]); acc[1] = fmaf(wv, lo.y, acc[1]); acc[2] = fmaf(wv, lo.z, acc[2]); acc[3] = fmaf(wv, lo.w, acc[3]);
        acc[4] = fmaf(wv, hi.x, acc[4]); acc[5] = fmaf(wv, hi.y, acc[5]); acc[6] = fmaf(wv, hi.z, acc[6]); acc[7] = fmaf(wv, hi.w, acc[7]);
    };
    if (vec) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
            if ((c * 4 + sub) * 8 < rank)
#pragma unroll
                for (int u = 0; u < 8; ++u) add(first[c][u], (c * 4 + sub) * 8 + u);
        for (int r = (8 + sub) * 8; r < rank; r += 32) {
            float wv[8];
            load4(wr + r, wv);
            load4(wr + r + 4, wv + 4);
#pragma unroll
            for (int u = 0; u < 8; ++u) add(wv[u], r + u);
        }
    } else {
        for (int r = sub; r < rank; r += 4) add(to_f32(wr[r]), r);
    }
#pragma unroll
    for (int tt = 0; tt < LR_TOK; ++tt) {
        acc[tt] += __shfl_xor_sync(0xffffffffu, acc[tt], 1);
        acc[tt] += __shfl_xor_sync(0xffffffffu, acc[tt], 2);
    }
    if (row >= n) return;
    float* o = out + (size_t)t0 * ld_out + (second ? p.n0 : 0) + row;
#pragma unroll
    for (int tt = 0; tt < LR_TOK; ++tt)
        if ((tt & 3) == sub && t0 + tt < T) o[(size_t)tt * ld_out] = acc[tt];
}
}  // namespace

extern "C" int rb_delta_prep(const void* in, int in_dtype, int n_in, long long in_stride, int row_stride, int q_off, int k_off,
                             int v_off, int b_off, int heads, int kv_heads, int dim, int vdim, int taps, const float* conv_w,
                             float* kept, const void* z, int z_dtype, int z_n_in, long long z_in_stride, int z_row_stride,
                             const float* dt_bias, const float* a_log, int per_channel, float unit_eps, float q_scale,
                             const int* seq_slot, const int* cu_q, int n_seqs, int max_q_len, float* u, int ld_u, int uq, int uk,
                             int uv, int ug, int ub, int ud, void* stream) {
    if (n_seqs <= 0 || max_q_len <= 0) return RB_OK;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || n_in < 1 || z_n_in < 1 || n_seqs > 65535 ||
        taps < 1 || taps > PREP_MAX_TAPS || (taps > 1 && !kept))
        return RB_ERR_BAD_SIZE;
    const PrepArgs a{(size_t)in_stride, n_in, row_stride, q_off, k_off, v_off, b_off, heads, kv_heads, dim, vdim, taps,
                     2 * kv_heads * dim + heads * vdim, conv_w, kept, (size_t)z_in_stride, z_n_in, z_row_stride, dt_bias, a_log,
                     per_channel, unit_eps, q_scale, seq_slot, cu_q, u, ld_u, uq, uk, uv, ug, ub, ud};
    const dim3 grid(kv_heads + heads, (max_q_len + PREP_TOK - 1) / PREP_TOK, n_seqs);
    if (grid.y > 65535) return RB_ERR_BAD_SIZE;
    const dim3 block(max_q_len == 1 ? 32 : 128);
    const size_t isz = in_dtype == RB_F32 ? 4 : 2, zsz = z_dtype == RB_F32 ? 4 : 2;
    const bool vec = ((dim | vdim | row_stride | q_off | k_off | v_off | ld_u | uq | uk | uv) & 3) == 0 && (in_stride & 3) == 0 &&
                     ((uintptr_t)in & (4 * isz - 1)) == 0 && (((uintptr_t)u | (uintptr_t)conv_w | (uintptr_t)kept) & 15) == 0 &&
                     (!per_channel || (((ug | z_row_stride) & 3) == 0 && (z_in_stride & 3) == 0 && ((uintptr_t)z & (4 * zsz - 1)) == 0 &&
                                       ((uintptr_t)dt_bias & 15) == 0));
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
    const bool rows = vec && n_in == 1 && z_n_in == 1 && max_q_len > 1 && taps <= 4 && dim <= 128 && vdim <= 128;
#define RB_DP(IT, ZT)                                                                                          \
    do {                                                                                                       \
        if (rows && taps == 4) RB_LAUNCH((delta_prep_rows_kernel<IT, ZT, 4>), grid, block, 0, s, (const IT*)in, (const ZT*)z, a);      \
        else if (rows && taps == 3) RB_LAUNCH((delta_prep_rows_kernel<IT, ZT, 3>), grid, block, 0, s, (const IT*)in, (const ZT*)z, a); \
        else if (rows && taps == 2) RB_LAUNCH((delta_prep_rows_kernel<IT, ZT, 2>), grid, block, 0, s, (const IT*)in, (const ZT*)z, a); \
        else if (vec) RB_LAUNCH((delta_prep_kernel<IT, ZT, 4>), grid, block, 0, s, (const IT*)in, (const ZT*)z, a); \
        else RB_LAUNCH((delta_prep_kernel<IT, ZT, 1>), grid, block, 0, s, (const IT*)in, (const ZT*)z, a);     \
    } while (0)
    if (in_dtype == RB_F32 && z_dtype == RB_F32) RB_DP(float, float);
    else if (in_dtype == RB_BF16 && z_dtype == RB_F32) RB_DP(bf, float);
    else if (in_dtype == RB_BF16 && z_dtype == RB_BF16) RB_DP(bf, bf);
    else return RB_ERR_BAD_DTYPE;
#undef RB_DP
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_delta_scan(const float* u, int ld_u, int uq, int uk, int uv, int ug, int ub, int ud, int heads, int kv_heads,
                             int dim, int vdim, int per_channel, float* state, const int* seq_slot, const int* cu_q, int n_seqs,
                             float* out, int ld_out, void* stream) {
    if (n_seqs <= 0) return RB_OK;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || n_seqs > 65535 || heads > 65535)
        return RB_ERR_BAD_SIZE;
    if ((dim & 3) == 0 && ((uintptr_t)state & 15)) return RB_ERR_BAD_ALIGN;
    ScanArgs a{u, ld_u, uq, uk, uv, ug, ub, ud, heads, kv_heads, dim, vdim, state, seq_slot, cu_q, out, ld_out, 0};
    a.vec = ((dim | vdim | ld_u | uq | uk | uv) & 3) == 0 && (!per_channel || (ug & 3) == 0) && ((uintptr_t)u & 15) == 0;
    cudaStream_t s = (cudaStream_t)stream;
#define RB_DS(R4, TB) return per_channel ? launch_scan<R4, true, TB>(a, n_seqs, s) : launch_scan<R4, false, TB>(a, n_seqs, s)
    if (dim <= 64) RB_DS(1, 16);
    if (dim <= 128) RB_DS(2, 16);
    if (dim <= 256) RB_DS(4, 8);
    if (dim <= 512) RB_DS(8, 4);
#undef RB_DS
    return RB_ERR_BAD_SIZE;
}

extern "C" int rb_low_rank(const void* in, int in_dtype, int n_in, long long in_stride, int row_stride, int x_off0, int rank0,
                           const void* w0, int n0, int x_off1, int rank1, const void* w1, int n1, int w_dtype, int T, float* out,
                           int ld_out, void* stream) {
    if (T <= 0) return RB_OK;
    if (rank0 <= 0 || n0 <= 0 || n_in < 1 || n1 < 0 || (n1 > 0 && rank1 <= 0)) return RB_ERR_BAD_SIZE;
    const int rank = n1 > 0 && rank1 > rank0 ? rank1 : rank0;
    const size_t smem = (size_t)((rank + 7) / 8) * 72 * sizeof(float);
    if (smem > 48 * 1024) return RB_ERR_BAD_SIZE;
    const LowRank p{w0, w1, x_off0, rank0, n0, x_off1, rank1, n1};
    const dim3 grid((n0 + LR_ROWS - 1) / LR_ROWS + (n1 + LR_ROWS - 1) / LR_ROWS, (T + LR_TOK - 1) / LR_TOK);
    if (grid.y > 65535) return RB_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    typedef __nv_bfloat16 bf;
#define RB_LR(IT, WT) RB_LAUNCH((low_rank_kernel<IT, WT>), grid, dim3(4 * LR_ROWS), smem, s, (const IT*)in, n_in, (size_t)in_stride, row_stride, p, T, out, ld_out)
    if (in_dtype == RB_F32 && w_dtype == RB_BF16) RB_LR(float, bf);
    else if (in_dtype == RB_F32 && w_dtype == RB_F32) RB_LR(float, float);
    else if (in_dtype == RB_BF16 && w_dtype == RB_BF16) RB_LR(bf, bf);
    else if (in_dtype == RB_BF16 && w_dtype == RB_F32) RB_LR(bf, float);
    else return RB_ERR_BAD_DTYPE;
#undef RB_LR
    RB_LAUNCH_CHECK();
    return RB_OK;
}

// The same for prompts, four tokens at a time: vecs float32 [heads][T][3][dimp] and firsts float32 [heads][n_chunks][dimp + 36] are
// work space, n_chunks >= T / 4 + n_seqs, dimp = dim rounded up to 64 (128, 256).  RB_ERR_BAD_SIZE for dim > 256.
extern "C" int rb_delta_scan_chunks(const float* u, int ld_u, int uq, int uk, int uv, int ug, int ub, int ud, int heads, int kv_heads,
                                    int dim, int vdim, int per_channel, float* state, const int* seq_slot, const int* cu_q, int n_seqs,
                                    int max_q_len, int T, float* vecs, float* firsts, int n_chunks, int dimp, float* out, int ld_out,
                                    void* stream) {
    (void)ud;
    if (n_seqs <= 0 || max_q_len <= 0) return RB_OK;
    if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || dim <= 0 || vdim <= 0 || n_seqs > 65535 || heads > 65535 || dim > dimp ||
        (dimp != 64 && dimp != 128 && dimp != 256))
        return RB_ERR_BAD_SIZE;
    if (T <= 0 || n_chunks < T / CH_T + n_seqs) return RB_ERR_BAD_SIZE;
    if (((uintptr_t)vecs | (uintptr_t)firsts) & 15) return RB_ERR_BAD_ALIGN;
    cudaStream_t s = (cudaStream_t)stream;
    RB_LAUNCH((delta_chunk_kernel), dim3((max_q_len + 4 * CH_T - 1) / (4 * CH_T), heads, n_seqs), dim3(128), 0, s, u, ld_u, uq, uk, ug, ub,
              heads, kv_heads, dim, dimp, per_channel, seq_slot, cu_q, T, n_chunks, vecs, firsts);
    RB_LAUNCH_CHECK();
    ChunkArgs a{u, vecs, firsts, T, n_chunks, ld_u, uv, heads, dim, vdim, dimp, state, seq_slot, cu_q, out, ld_out, 0};
    a.vec = ((vdim | ld_u | uv) & 3) == 0 && ((uintptr_t)u & 15) == 0;
    // more blocks than three a multiprocessor: a shorter batch of tokens, so that four fit
    const bool many = (long long)n_seqs * heads * ((vdim + 15) / 16) > 3 * 148;
    if (dimp == 64) return many ? launch_chunks<1, 8>(a, n_seqs, s) : launch_chunks<1, 16>(a, n_seqs, s);
    if (dimp == 128) return many ? launch_chunks<2, 8>(a, n_seqs, s) : launch_chunks<2, 16>(a, n_seqs, s);
    return launch_chunks<4, 8>(a, n_seqs, s);
}
