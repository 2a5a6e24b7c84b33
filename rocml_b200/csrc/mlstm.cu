// A matrix memory with exponential gates and a running maximum (mLSTM), per (sequence, head):
//
//   i = cap * tanh(zi / cap),  f = log sigmoid(cap * tanh(zf / cap))            log gates, one a head
//   m_t = max(f + m_(t-1), i)                                                    starts at 0
//   S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T                      S [dim, vdim], 32-bit
//   n_t = the same with k alone                                                  n [dim]
//   o_t = S_t^T q / (max(|n_t . q|, e^(-m_t)) + eps)
//
// The kernels write S^T q and the divisor apart; what follows (a norm per head, the output gate) divides.  The state of a
// slot: S [heads][dim][vdim], n [heads][dim], and m [heads][2], of which the token at position p writes entry p & 1 and
// reads the other: the blocks that share a head in a decode step then never read what one of them writes.
//
//   mlstm_gates   a step's log gates for all tokens of a sequence and head: the running maximum is a scan of pairs
//                 (f, i) -> m' = max(f + m, i); out come log keep = f + m_(t-1) - m_t <= 0, log add = i - m_t <= 0 and
//                 e^(-m_t), and the slot's m moves on.
//   mlstm_step    one token a sequence: the state streams through registers (a warp every eighth row, a lane a column),
//                 read, decayed, updated and written once; one more block a head does n, the divisor and m.
//   mlstm blocks  prompts, by blocks of 64 tokens side by side.  With c_t the sum of log keep inside a block that
//                 starts from (S0, n0):
//                   S_t^T q_t = e^(c_t) S0^T q_t + sum_{s <= t} e^(c_t - c_s + log add_s) (q_t . k_s) v_s     (n: v = 1)
//                   S_end = e^(c_end) S0 + sum_s e^(c_end - c_s + log add_s) k_s v_s^T
//                 every exponent is <= 0.  Four kernels: the decayed scores of every block; every block's own sum; the
//                 states the blocks start from, along each sequence; every block's results.  c is kept as two floats, so
//                 that a difference of two large sums is as exact as a small one.
//
//   mlstm chain   the same blocks for bfloat16 projections on the tensor cores (mma.sync), without the states in between going
//                 through memory: a thread block owns 32 of a head's columns and walks the sequence's blocks of tokens with its
//                 part of the state in registers; one more block a head does n and the divisors.  32-bit numbers enter a product as
//                 the sum of three bfloat16 numbers (24 bits), their partner there being bfloat16 as it came from the
//                 projection, so that every product is that of the 32-bit numbers, with 32-bit sums.  A kernel before it forms
//                 the decayed scores (as three planes) and the decays for all blocks at once.
//
// All arithmetic is 32-bit.  q, k, v are columns of the layer's projection, in the activations' type or as 32-bit partial
// sums that are added first; the gates' columns are 32-bit always.
#include "common.cuh"
#include "mma_tiles.cuh"
#include "api.h"

using namespace rb;

namespace {
constexpr int CB = 64;              // tokens a block
constexpr int CT = 256;             // threads: a 16 x 16 grid, each thread a 4 x 4 tile of a 64 x 64 result
constexpr int CL = CB + 4;          // row length of transposed tiles (a multiple of 4 that is no multiple of 32)

// Columns of the step's projection rows: `n_in` partial sums of [T][row_stride], added in order.
template <typename IT>
struct Cols {
    const IT* p;
    int n_in;
    size_t in_stride;
    int row_stride;
    __device__ __forceinline__ float operator()(int t, int col) const {
        const int cols[1] = {col};
        float v[1];
        many<1>(t, cols, v);
        return v[0];
    }
    // N columns at a time: four partial sums of each in flight, added in order
    template <int N>
    __device__ __forceinline__ void many(int t, const int (&col)[N], float (&v)[N]) const {
        const IT* x = p + (size_t)t * row_stride;
#pragma unroll
        for (int e = 0; e < N; ++e) v[e] = to_f32(x[col[e]]);
        for (int s = 1; s < n_in; s += 4) {
            float y[4][N];
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < N; ++e) y[j][e] = s + j < n_in ? to_f32(x[(size_t)(s + j) * in_stride + col[e]]) : 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < N; ++e) v[e] += y[j][e];
        }
    }
};

__device__ __forceinline__ float capped_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// One block a (head, sequence), a thread a token, as many tokens at a time as the block has threads.
__global__ void __launch_bounds__(1024)
mlstm_gates_kernel(const Cols<float> g, int i_off, int f_off, float cap, int heads, float* __restrict__ m_state,
                   const int* __restrict__ seq_slot, const int* __restrict__ cu_q, const int* __restrict__ positions, int T,
                   float* __restrict__ log_keep, float* __restrict__ log_add, float* __restrict__ em) {
    pdl_trigger();
    pdl_wait();
    __shared__ float wf[32], wm[32], m_carry;
    const int h = blockIdx.x, b = blockIdx.y;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
    if (n <= 0) return;
    const int pos0 = positions[t0];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float* mine = m_state + ((size_t)slot * heads + h) * 2;
    float m = mine[(pos0 + 1) & 1];
    for (int base = 0; base < n; base += blockDim.x) {
        const int t = base + threadIdx.x;
        const bool here = t < n;
        float i = -INFINITY, f = 0.f;                       // past the end: the pair that changes nothing
        if (here) {
            i = capped_gate(g(t0 + t, i_off + h), cap);
            f = log_sigmoid(capped_gate(g(t0 + t, f_off + h), cap));
        }
        float F = f, M = i;                                 // the pair of all tokens up to this one
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fp = __shfl_up_sync(0xffffffffu, F, o), Mp = __shfl_up_sync(0xffffffffu, M, o);
            if (lane >= o) { M = fmaxf(Mp + F, M); F += Fp; }
        }
        if (lane == 31) { wf[warp] = F; wm[warp] = M; }
        __syncthreads();
        float start = m;                                    // the maximum before this warp's first token
        for (int w = 0; w < warp; ++w) start = fmaxf(wf[w] + start, wm[w]);
        const float m_t = fmaxf(F + start, M);
        float m_prev = __shfl_up_sync(0xffffffffu, m_t, 1);
        if (lane == 0) m_prev = start;
        if (here) {
            const size_t at = (size_t)h * T + t0 + t;
            log_keep[at] = fminf(f + m_prev - m_t, 0.f);
            log_add[at] = fminf(i - m_t, 0.f);
            em[at] = expf(-m_t);
        }
        if (warp == nw - 1 && lane == 31) m_carry = m_t;
        __syncthreads();
        m = m_carry;
    }
    if (threadIdx.x == 0) mine[(pos0 + n - 1) & 1] = m;
}

// ---- one token a sequence -------------------------------------------------------------------------------------------
template <typename IT, int V>
__global__ void __launch_bounds__(256, 3)
mlstm_step_kernel(const Cols<IT> x, int q_off, int k_off, int v_off, const Cols<float> g, int i_off, int f_off, float cap,
                  float q_scale, float eps, int heads, int dim, int vdim, float* __restrict__ S_state, float* __restrict__ n_state,
                  float* __restrict__ m_state, const int* __restrict__ seq_slot, const int* __restrict__ cu_q,
                  const int* __restrict__ positions, float* __restrict__ out, int ld_out, float* __restrict__ den) {
    pdl_trigger();
    pdl_wait();
    constexpr int LPR = 32 / V, RG = 256 / LPR, R = 8;      // threads a row of 32 columns, rows side by side, rows in flight a thread
    extern __shared__ __align__(16) float sm[];
    __shared__ float part[8][32];
    __shared__ float red[33];
    float* qs = sm;            // [dim]
    float* ks = sm + dim;      // [dim], times e^(i - m)
    const int b = blockIdx.z, h = blockIdx.y;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    const int t = cu_q[b];
    if (cu_q[b + 1] <= t) return;
    const bool last = blockIdx.x == gridDim.x - 1;          // this block does n, the divisor and m
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int col = (threadIdx.x % LPR) * V, j = blockIdx.x * 32 + col, r0 = threadIdx.x / LPR;
    const bool mine_cols = !last && j < vdim;               // (V divides vdim)
    float* S = S_state + (((size_t)slot * heads + h) * dim) * vdim + j;
    float s[R][V];
    auto ask = [&](int base) {
#pragma unroll
        for (int u = 0; u < R; ++u) {
            const int c = base + r0 + u * RG;
            if (c < dim) {
                if constexpr (V == 4) *reinterpret_cast<float4*>(s[u]) = *reinterpret_cast<const float4*>(S + (size_t)c * vdim);
                else s[u][0] = S[(size_t)c * vdim];
            }
        }
    };
    if (mine_cols) ask(0);                                  // the state travels while the gates are formed
    const int pos = positions[t];
    float* mine = m_state + ((size_t)slot * heads + h) * 2;
    const float m0 = mine[(pos + 1) & 1];
    const int gate_cols[2] = {i_off + h, f_off + h};
    float gate[2];
    g.template many<2>(t, gate_cols, gate);
    // q, k and v of the first pass together (a column past the end stands for the last one)
    const int c_first = min((int)threadIdx.x, dim - 1), j_first = mine_cols ? j : 0;
    int row_cols[2 + V];
    float row[2 + V];
    row_cols[0] = q_off + h * dim + c_first; row_cols[1] = k_off + h * dim + c_first;
#pragma unroll
    for (int e = 0; e < V; ++e) row_cols[2 + e] = v_off + h * vdim + j_first + e;
    x.template many<2 + V>(t, row_cols, row);
    const float i = capped_gate(gate[0], cap), f = log_sigmoid(capped_gate(gate[1], cap));
    const float m1 = fmaxf(f + m0, i);
    const float keep = expf(f + m0 - m1), add = expf(i - m1);
    if (threadIdx.x < dim) {
        qs[threadIdx.x] = row[0] * q_scale;
        ks[threadIdx.x] = row[1] * add;
    }
    for (int c = threadIdx.x + 256; c < dim; c += 256) {
        qs[c] = x(t, q_off + h * dim + c) * q_scale;
        ks[c] = x(t, k_off + h * dim + c) * add;
    }
    const float* v = row + 2;
    __syncthreads();
    if (last) {
        float* n = n_state + ((size_t)slot * heads + h) * dim;
        float acc = 0.f;
        for (int c = threadIdx.x; c < dim; c += 256) {
            const float w = fmaf(keep, n[c], ks[c]);
            n[c] = w;
            acc = fmaf(w, qs[c], acc);
        }
        acc = block_sum(acc, red);
        if (threadIdx.x == 0) {
            den[(size_t)t * heads + h] = fmaxf(fabsf(acc), expf(-m1)) + eps;
            mine[pos & 1] = m1;
        }
        return;
    }
    float acc[V] = {};
    if (mine_cols) {
        for (int base = 0;;) {
#pragma unroll
            for (int u = 0; u < R; ++u) {
                const int c = base + r0 + u * RG;
                if (c < dim) {
#pragma unroll
                    for (int e = 0; e < V; ++e) {
                        s[u][e] = fmaf(ks[c], v[e], keep * s[u][e]);
                        acc[e] = fmaf(s[u][e], qs[c], acc[e]);
                    }
                    if constexpr (V == 4) *reinterpret_cast<float4*>(S + (size_t)c * vdim) = *reinterpret_cast<const float4*>(s[u]);
                    else S[(size_t)c * vdim] = s[u][0];
                }
            }
            base += R * RG;
            if (base >= dim) break;
            ask(base);
        }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
#pragma unroll
        for (int o = LPR; o < 32; o <<= 1) acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], o);
        if (lane < LPR) part[warp][col + e] = acc[e];
    }
    __syncthreads();
    const int jo = blockIdx.x * 32 + lane;
    if (warp == 0 && jo < vdim) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w][lane];
        out[(size_t)t * ld_out + (size_t)h * vdim + jo] = o;
    }
}

// ---- prompts: blocks of 64 tokens side by side ---------------------------------------------------------------------------
// Which sequence and which of its blocks of tokens the grid's block `g` is (blocks are numbered sequence after sequence).
__device__ __forceinline__ bool find_tokens(int g, const int* seq_slot, const int* cu_q, int n_seqs, int* t0, int* m) {
    int base = 0;
    for (int b = 0; b < n_seqs; ++b) {
        const int n = cu_q[b + 1] - cu_q[b];
        const int nb = seq_slot[b] >= 0 ? (n + CB - 1) / CB : 0;
        if (g < base + nb) {
            const int c = g - base;
            *t0 = cu_q[b] + c * CB; *m = min(CB, n - c * CB);
            return true;
        }
        base += nb;
    }
    return false;
}

// The running sums of log keep inside a block, as two floats each (hi + lo), and the block's log add; rows past m repeat
// the last sum and add nothing.
struct BlockGates {
    float hi[CB], lo[CB], add[CB];
    __device__ __forceinline__ float decay(int t, int s) const { return (hi[t] - hi[s]) + (lo[t] - lo[s]); }   // c_t - c_s
};
__device__ __forceinline__ void block_gates(BlockGates& g, const float* log_keep, const float* log_add, int t0, int m) {
    const int t = threadIdx.x;
    if (t < CB) {
        g.hi[t] = t < m ? log_keep[t0 + t] : 0.f;
        g.add[t] = t < m ? log_add[t0 + t] : -INFINITY;
    }
    __syncthreads();
    double c = 0.0;
    if (t < CB)
        for (int r = 0; r <= t; ++r) c += (double)g.hi[r];
    __syncthreads();
    if (t < CB) {
        g.hi[t] = (float)c;
        g.lo[t] = (float)(c - (double)(float)c);
    }
    __syncthreads();
}

// acc[4][4] += A^T[k][rows] . B[k][cols] over k < K: At is [K][lda] (the thread's rows at 4 * ty), Bm is [K][ldb].
__device__ __forceinline__ void tile_mm(float (&acc)[4][4], const float* At, int lda, const float* Bm, int ldb, int K, int ty, int tx) {
#pragma unroll 4
    for (int k = 0; k < K; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(At + k * lda + 4 * ty);
        const float4 b = *reinterpret_cast<const float4*>(Bm + k * ldb + 4 * tx);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
}

// (0) the decayed scores of a block, stored [s][t]: e^(c_t - c_s + log add_s) (q_t . k_s) for s <= t; and their sums over s.
template <typename IT>
__global__ void __launch_bounds__(CT)
mlstm_block_scores_kernel(const Cols<IT> x, int q_off, int k_off, float q_scale, int heads, int dim, const float* __restrict__ log_keep,
                          const float* __restrict__ log_add, int T, const int* __restrict__ seq_slot, const int* __restrict__ cu_q,
                          int n_seqs, float* __restrict__ scores, float* __restrict__ den) {
    pdl_trigger();
    pdl_wait();
    __shared__ __align__(16) float Qt[CB * CL];
    __shared__ __align__(16) float Kt[CB * CL];
    __shared__ BlockGates g;
    int t0, m;
    if (!find_tokens(blockIdx.y, seq_slot, cu_q, n_seqs, &t0, &m)) return;
    const int h = blockIdx.x;
    block_gates(g, log_keep + (size_t)h * T, log_add + (size_t)h * T, t0, m);
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    float acc[4][4] = {};
    for (int n0 = 0; n0 < dim; n0 += CB) {
        __syncthreads();
        for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
            const int s = idx / CB, i = idx - s * CB;         // consecutive threads read consecutive dimensions of one token
            const bool in = s < m && n0 + i < dim;
            Qt[i * CL + s] = in ? x(t0 + s, q_off + h * dim + n0 + i) * q_scale : 0.f;
            Kt[i * CL + s] = in ? x(t0 + s, k_off + h * dim + n0 + i) : 0.f;
        }
        __syncthreads();
        tile_mm(acc, Kt, CL, Qt, CL, min(CB, dim - n0), ty, tx);            // rows s, columns t
    }
    __syncthreads();
    float* dst = scores + ((size_t)blockIdx.y * heads + h) * CB * CB;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int s = 4 * ty + i;
        float o[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = 4 * tx + j;
            o[j] = s <= t && t < m ? acc[i][j] * expf(g.decay(t, s) + g.add[s]) : 0.f;
            Qt[s * CL + t] = o[j];
        }
        *reinterpret_cast<float4*>(dst + s * CB + 4 * tx) = make_float4(o[0], o[1], o[2], o[3]);
    }
    __syncthreads();
    if (threadIdx.x < m) {
        float sum = 0.f;
        for (int s = 0; s <= (int)threadIdx.x; ++s) sum += Qt[s * CL + threadIdx.x];
        den[(size_t)(t0 + threadIdx.x) * heads + h] = sum;
    }
}

// (1) every block's own sum: sum_s e^(c_end - c_s + log add_s) k_s [v_s | 1]^T, and e^(c_end).
template <typename IT>
__global__ void __launch_bounds__(CT)
mlstm_block_sum_kernel(const Cols<IT> x, int k_off, int v_off, int heads, int dim, int vdim, const float* __restrict__ log_keep,
                       const float* __restrict__ log_add, int T, const int* __restrict__ seq_slot, const int* __restrict__ cu_q,
                       int n_seqs, float* __restrict__ work, float* __restrict__ work_n, float* __restrict__ block_decay) {
    pdl_trigger();
    pdl_wait();
    __shared__ __align__(16) float Kw[CB * CB];       // [s][dim]: k_s times its weight
    __shared__ __align__(16) float Vs[CB * CB];       // [s][vdim]
    __shared__ BlockGates g;
    __shared__ float w[CB];
    int t0, m;
    if (!find_tokens(blockIdx.z, seq_slot, cu_q, n_seqs, &t0, &m)) return;
    const int h = blockIdx.y, p0 = blockIdx.x * CB;
    block_gates(g, log_keep + (size_t)h * T, log_add + (size_t)h * T, t0, m);
    if (threadIdx.x == 0 && blockIdx.x == 0) block_decay[(size_t)blockIdx.z * heads + h] = expf(g.hi[m - 1] + g.lo[m - 1]);
    if (threadIdx.x < CB) w[threadIdx.x] = (int)threadIdx.x < m ? expf(g.decay(m - 1, threadIdx.x) + g.add[threadIdx.x]) : 0.f;
    for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
        const int s = idx / CB, j = idx - s * CB;
        Vs[idx] = s < m && p0 + j < vdim ? x(t0 + s, v_off + h * vdim + p0 + j) : 0.f;
    }
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const size_t at = (size_t)blockIdx.z * heads + h;
    for (int n0 = 0; n0 < dim; n0 += CB) {
        __syncthreads();
        for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
            const int s = idx / CB, i = idx - s * CB;
            Kw[idx] = s < m && n0 + i < dim ? x(t0 + s, k_off + h * dim + n0 + i) * w[s] : 0.f;
        }
        __syncthreads();
        float acc[4][4] = {};
        tile_mm(acc, Kw, CB, Vs, CB, m, ty, tx);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int row = n0 + 4 * ty + i, col = p0 + 4 * tx + j;
                if (row < dim && col < vdim) work[(at * dim + row) * vdim + col] = acc[i][j];
            }
        if (blockIdx.x == 0 && threadIdx.x < CB && n0 + (int)threadIdx.x < dim) {
            float sum = 0.f;
            for (int s = 0; s < m; ++s) sum += Kw[s * CB + threadIdx.x];
            work_n[at * dim + n0 + threadIdx.x] = sum;
        }
    }
}

// (2) along each sequence: the state every block starts from takes the place of the block's own sum; the slot receives the
// state after the last block.  Elementwise over [S | n]; eight blocks' sums in flight.
__global__ void __launch_bounds__(256)
mlstm_block_states_kernel(float* __restrict__ work, float* __restrict__ work_n, const float* __restrict__ block_decay,
                          float* __restrict__ S_state, float* __restrict__ n_state, int heads, int dim, int vdim,
                          const int* __restrict__ seq_slot, const int* __restrict__ cu_q) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.z, h = blockIdx.y;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    int first = 0;
    for (int i = 0; i < b; ++i) first += seq_slot[i] >= 0 ? (cu_q[i + 1] - cu_q[i] + CB - 1) / CB : 0;
    const int nb = (cu_q[b + 1] - cu_q[b] + CB - 1) / CB;
    if (nb <= 0) return;
    const int np = dim * vdim;
    int e = blockIdx.x * 256 + threadIdx.x;
    if (e >= np + dim) return;
    float* st;
    float* wk;
    size_t stride;
    if (e < np) {
        stride = (size_t)heads * np;
        st = S_state + ((size_t)slot * heads + h) * np + e;
        wk = work + ((size_t)first * heads + h) * np + e;
    } else {
        e -= np;
        stride = (size_t)heads * dim;
        st = n_state + ((size_t)slot * heads + h) * dim + e;
        wk = work_n + ((size_t)first * heads + h) * dim + e;
    }
    float S = *st;
    for (int c0 = 0; c0 < nb; c0 += 8) {
        float own[8], dec[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            own[j] = c0 + j < nb ? wk[(size_t)(c0 + j) * stride] : 0.f;
            dec[j] = c0 + j < nb ? block_decay[(size_t)(first + c0 + j) * heads + h] : 1.f;
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (c0 + j < nb) {
                wk[(size_t)(c0 + j) * stride] = S;
                S = fmaf(dec[j], S, own[j]);
            }
        }
    }
    *st = S;
}

// (3) every block's results: e^(c_t) S0^T q_t + sum_s scores[s][t] v_s, and (first column tile) the divisors.
template <typename IT>
__global__ void __launch_bounds__(CT)
mlstm_block_out_kernel(const Cols<IT> x, int q_off, int v_off, float q_scale, float eps, int heads, int dim, int vdim,
                       const float* __restrict__ log_keep, const float* __restrict__ log_add, const float* __restrict__ em, int T,
                       const int* __restrict__ seq_slot, const int* __restrict__ cu_q, int n_seqs, const float* __restrict__ work,
                       const float* __restrict__ work_n, const float* __restrict__ scores, float* __restrict__ out, int ld_out,
                       float* __restrict__ den) {
    pdl_trigger();
    pdl_wait();
    __shared__ __align__(16) float Qt[CB * CL];       // [dim][t]; later the scores [s][t]
    __shared__ __align__(16) float Bs[CB * CB];       // the starting state [dim][vdim]; later v [s][vdim]
    __shared__ BlockGates g;
    int t0, m;
    if (!find_tokens(blockIdx.z, seq_slot, cu_q, n_seqs, &t0, &m)) return;
    const int h = blockIdx.y, p0 = blockIdx.x * CB;
    block_gates(g, log_keep + (size_t)h * T, log_add + (size_t)h * T, t0, m);
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const size_t at = (size_t)blockIdx.z * heads + h;
    float acc[4][4] = {};
    float nq = 0.f;
    for (int n0 = 0; n0 < dim; n0 += CB) {
        __syncthreads();
        const int rows = min(CB, dim - n0);
        for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
            const int s = idx / CB, i = idx - s * CB;
            Qt[i * CL + s] = s < m && i < rows ? x(t0 + s, q_off + h * dim + n0 + i) * q_scale : 0.f;
        }
        for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
            const int i = idx / CB, j = idx - i * CB;
            Bs[idx] = i < rows && p0 + j < vdim ? work[(at * dim + n0 + i) * vdim + p0 + j] : 0.f;
        }
        __syncthreads();
        tile_mm(acc, Qt, CL, Bs, CB, rows, ty, tx);           // rows t, columns vdim
        if (blockIdx.x == 0 && (int)threadIdx.x < m)
            for (int i = 0; i < rows; ++i) nq = fmaf(Qt[i * CL + threadIdx.x], work_n[at * dim + n0 + i], nq);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        const float e = t < m ? expf(g.hi[t] + g.lo[t]) : 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] *= e;
    }
    if (blockIdx.x == 0 && (int)threadIdx.x < m) {
        const int t = threadIdx.x;
        float* d = den + (size_t)(t0 + t) * heads + h;
        *d = fmaxf(fabsf(fmaf(expf(g.hi[t] + g.lo[t]), nq, *d)), em[(size_t)h * T + t0 + t]) + eps;
    }
    __syncthreads();
    const float* sc = scores + at * CB * CB;
    for (int idx = threadIdx.x; idx < CB * CB; idx += CT) {
        const int s = idx / CB, j = idx - s * CB;
        Qt[s * CL + j] = sc[idx];
        Bs[idx] = s < m && p0 + j < vdim ? x(t0 + s, v_off + h * vdim + p0 + j) : 0.f;
    }
    __syncthreads();
    tile_mm(acc, Qt, CL, Bs, CB, m, ty, tx);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        if (t >= m) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int col = p0 + 4 * tx + j;
            if (col < vdim) out[(size_t)(t0 + t) * ld_out + (size_t)h * vdim + col] = acc[i][j];
        }
    }
}

// ---- prompts on the tensor cores --------------------------------------------------------------------------------------------
using namespace mma_tiles;
typedef __nv_bfloat16 bf16;

// x = hi + mid + lo in bfloat16, two neighbouring numbers packed
__device__ __forceinline__ void split3(float x, float y, uint32_t (&p)[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
        p[i] = *reinterpret_cast<const uint32_t*>(&h);
        const float2 f = __bfloat1622float2(h);
        x -= f.x;
        y -= f.y;
    }
}

struct Rows16 {            // bfloat16 projection rows
    const bf16* p;
    long long stride;
};

constexpr int PLANE = CB * CB;      // one plane of a block's decayed scores

// The decayed scores of a block as three planes [3][t][s], their sums over s, and for every token e^(c_t) * q_scale (`ec`) and
// e^(c_end - c_t + log add_t) (`wt`), [heads][T]; e^(c_end) per block and head.  A warp owns 16 tokens t.
template <int DIM>
__global__ void __launch_bounds__(128)
mlstm_scores_tc_kernel(const Rows16 x, int q_off, int k_off, float q_scale, int heads, const float* __restrict__ log_keep,
                       const float* __restrict__ log_add, int T, const int* __restrict__ seq_slot, const int* __restrict__ cu_q, int n_seqs,
                       bf16* __restrict__ planes, float* __restrict__ ec, float* __restrict__ wt, float* __restrict__ block_decay,
                       float* __restrict__ den) {
    pdl_wait();         // (no early signal: the kernel after this one has few blocks that run long)
    extern __shared__ __align__(128) uint8_t raw_sm[];
    bf16* Qs = reinterpret_cast<bf16*>(raw_sm);        // [64][DIM]
    bf16* Ks = Qs + CB * DIM;
    __shared__ BlockGates g;
    int t0, m;
    if (!find_tokens(blockIdx.y, seq_slot, cu_q, n_seqs, &t0, &m)) return;
    const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    load_tile<DIM>(Qs, x.p + (long long)t0 * x.stride + q_off + h * DIM, x.stride, CB, m, threadIdx.x, 128);
    load_tile<DIM>(Ks, x.p + (long long)t0 * x.stride + k_off + h * DIM, x.stride, CB, m, threadIdx.x, 128);
    cp_async_commit();
    block_gates(g, log_keep + (size_t)h * T, log_add + (size_t)h * T, t0, m);
    if (threadIdx.x < m) {
        const int t = threadIdx.x;
        ec[(size_t)h * T + t0 + t] = expf(g.hi[t] + g.lo[t]) * q_scale;
        wt[(size_t)h * T + t0 + t] = expf(g.decay(m - 1, t) + g.add[t]);
    }
    if (threadIdx.x == 0) block_decay[(size_t)blockIdx.y * heads + h] = expf(g.hi[m - 1] + g.lo[m - 1]);
    cp_async_wait<0>();
    __syncthreads();
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const uint32_t qb = smem_addr(Qs), kb = smem_addr(Ks);
#pragma unroll 4
    for (int ks = 0; ks < DIM / 16; ++ks) {
        uint32_t a[4];
        ldmatrix_x4(tile_addr<DIM>(qb, warp * 16 + (lane & 15), ks * 2 + (lane >> 4)), a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int j = 0; j < 8; j += 2) {
            if (j * 8 > warp * 16 + 15) continue;                       // keys after this warp's last token
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(tile_addr<DIM>(kb, j * 8 + (lane & 7) + ((lane >> 4) & 1) * 8, ks * 2 + ((lane >> 3) & 1)), b0, b1, b2, b3);
            mma_bf16(acc[j], a, b0, b1);
            mma_bf16(acc[j + 1], a, b2, b3);
        }
    }
    bf16* dst = planes + ((size_t)blockIdx.y * heads + h) * 3 * PLANE;
    const int r0 = warp * 16 + (lane >> 2);
    float sum[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 8; ++j) {
        const int s = j * 8 + (lane & 3) * 2;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = r0 + 8 * r;
            float v[2];
#pragma unroll
            for (int e = 0; e < 2; ++e)
                v[e] = s + e <= t && t < m ? acc[j][2 * r + e] * q_scale * expf(g.decay(t, s + e) + g.add[s + e]) : 0.f;
            sum[r] += v[0] + v[1];
            uint32_t p[3];
            split3(v[0], v[1], p);
#pragma unroll
            for (int i = 0; i < 3; ++i) *reinterpret_cast<uint32_t*>(dst + i * PLANE + t * CB + s) = p[i];
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 1);
        sum[r] += __shfl_xor_sync(0xffffffffu, sum[r], 2);
        if ((lane & 3) == 0 && r0 + 8 * r < m) den[(size_t)(t0 + r0 + 8 * r) * heads + h] = sum[r];
    }
}

constexpr int CHAIN_COLS = 32;      // columns of the state a block owns
constexpr int RED_LD = 40;          // row length of the partial results (so that a half warp's pairs meet no bank twice)

template <int DIM>
struct ChainSizes {
    static constexpr int QK = CB * DIM * 2, V = CB * CHAIN_COLS * 2, P = 3 * PLANE * 2;
    static constexpr int BUF = 2 * QK + V + P;
    static constexpr int RED = 4 * CB * RED_LD * 4;
    static constexpr int SMEM = 2 * BUF + RED + 4 * CB * 4 + 128;
};

__device__ __forceinline__ uint32_t v_addr(uint32_t base, int row, int chunk) {       // rows of 64 bytes, four 16-byte chunks
    return base + (uint32_t)(row * 64 + ((chunk ^ ((row >> 1) & 3)) << 4));
}

// Warps: two groups of 16 columns times four quarters of the head's dimensions.  S^T (columns of S as rows of the tile) lives in
// the accumulators of its own update, which are at once the B operand of Q S.
template <int DIM>
__global__ void __launch_bounds__(256)
mlstm_chain_kernel(const Rows16 x, int q_off, int k_off, int v_off, float eps, int heads, int vdim, const bf16* __restrict__ planes,
                   const float* __restrict__ ec, const float* __restrict__ wt, const float* __restrict__ block_decay,
                   const float* __restrict__ em, int T, float* __restrict__ S_state, float* __restrict__ n_state,
                   const int* __restrict__ seq_slot, const int* __restrict__ cu_q, float* __restrict__ out, int ld_out,
                   float* __restrict__ den) {
    pdl_wait();
    using Z = ChainSizes<DIM>;
    extern __shared__ __align__(128) uint8_t raw_sm[];
    float* red = reinterpret_cast<float*>(raw_sm + 2 * Z::BUF);            // [4][64][RED_LD]
    float* tok = red + 4 * CB * RED_LD;                                    // [2 buffers][ec 64 | wt 64]
    const int h = blockIdx.y, b = blockIdx.z;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    const int t_begin = cu_q[b], n_tok = cu_q[b + 1] - t_begin;
    if (n_tok <= 0) return;
    int first = 0;
    for (int i = 0; i < b; ++i) first += seq_slot[i] >= 0 ? (cu_q[i + 1] - cu_q[i] + CB - 1) / CB : 0;
    const int nb = (n_tok + CB - 1) / CB;
    const bool n_role = blockIdx.x == gridDim.x - 1;
    const int p0 = blockIdx.x * CHAIN_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int grp = warp & 1, dq = warp >> 1;

    auto fetch = [&](int c) {
        uint8_t* buf = raw_sm + (c & 1) * Z::BUF;
        const int t0 = t_begin + c * CB, m = min(CB, n_tok - c * CB);
        const bf16* row = x.p + (long long)t0 * x.stride;
        load_tile<DIM>(reinterpret_cast<bf16*>(buf), row + q_off + h * DIM, x.stride, CB, m, tid, 256);
        load_tile<DIM>(reinterpret_cast<bf16*>(buf + Z::QK), row + k_off + h * DIM, x.stride, CB, m, tid, 256);
        if (!n_role) {
            uint8_t* vb = buf + 2 * Z::QK;
            {
                const int r = tid >> 2, ch = tid & 3;                       // 64 rows of four chunks
                cp_async16(vb + r * 64 + ((ch ^ ((r >> 1) & 3)) << 4),
                           row + (r < m ? (long long)r * x.stride : 0) + v_off + h * vdim + p0 + ch * 8, r < m);
            }
            const bf16* pl = planes + ((size_t)(first + c) * heads + h) * 3 * PLANE;
            load_tile<CB>(reinterpret_cast<bf16*>(vb + Z::V), pl, CB, 3 * CB, 3 * CB, tid, 256);
        }
        cp_async_commit();
    };
    // a token's two factors and the block's decay travel in registers until the block before them is done
    float next_tok = 0.f, next_decay = 0.f;
    auto ask = [&](int c) {
        const int t = tid & (CB - 1);
        next_decay = block_decay[(size_t)(first + c) * heads + h];
        if (tid < 2 * CB) next_tok = c * CB + t < n_tok ? (tid < CB ? ec : wt)[(size_t)h * T + t_begin + c * CB + t] : 0.f;
    };
    auto keep = [&](int c) {
        if (tid < 2 * CB) tok[(c & 1) * 2 * CB + tid] = next_tok;
    };
    ask(0);

    if (n_role) {
        // n and the divisors: a thread a dimension for the sums over tokens, a warp eight tokens for the products with q
        float* ns = red;
        float n = tid < DIM ? n_state[((size_t)slot * heads + h) * DIM + tid] : 0.f;
        fetch(0);
        keep(0);
        for (int c = 0; c < nb; ++c) {
            const float decay = next_decay;
            if (c + 1 < nb) { fetch(c + 1); ask(c + 1); cp_async_wait<1>(); }
            else cp_async_wait<0>();
            if (tid < DIM) ns[tid] = n;
            __syncthreads();
            const uint8_t* Q = raw_sm + (c & 1) * Z::BUF;
            const uint8_t* K = Q + Z::QK;
            const float* te = tok + (c & 1) * 2 * CB;
            const int t0 = t_begin + c * CB, m = min(CB, n_tok - c * CB);
            // eight tokens a warp, their sums side by side; lane u < 8 holds token u's divisor so far and its bound
            const int mine_t = warp + 8 * lane;
            float* dp = den + (size_t)(t0 + mine_t) * heads + h;
            const bool has = lane < 8 && mine_t < m;
            const float so_far = has ? *dp : 0.f, bound = has ? em[(size_t)h * T + t0 + mine_t] : 0.f;
            float acc[8] = {};
            for (int d = lane * 8; d < DIM; d += 256) {
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    const int row = warp + 8 * r;
                    const uint4 raw = *reinterpret_cast<const uint4*>(Q + row * DIM * 2 + (((d >> 3) ^ (row & 7)) << 4));
                    const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        acc[r] = fmaf(__uint_as_float(w[u] << 16), ns[d + 2 * u], acc[r]);
                        acc[r] = fmaf(__uint_as_float(w[u] & 0xFFFF0000u), ns[d + 2 * u + 1], acc[r]);
                    }
                }
            }
            float own = 0.f;
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                acc[r] = warp_sum(acc[r]);
                if (lane == r) own = acc[r];
            }
            if (has) *dp = fmaxf(fabsf(fmaf(te[mine_t], own, so_far)), bound) + eps;
            if (tid < DIM) {
                float sum = 0.f;
#pragma unroll 8
                for (int s = 0; s < CB; ++s)
                    sum = fmaf(te[CB + s], __bfloat162float(*reinterpret_cast<const bf16*>(K + s * DIM * 2 + (((tid >> 3) ^ (s & 7)) << 4) + (tid & 7) * 2)), sum);
                n = fmaf(decay, n, sum);
            }
            if (c + 1 < nb) keep(c + 1);
            __syncthreads();
        }
        if (tid < DIM) n_state[((size_t)slot * heads + h) * DIM + tid] = n;
        return;
    }

    constexpr int KS = DIM / 64;                 // k steps of 16 dimensions in a warp's quarter
    constexpr int NT = 2 * KS;                   // tiles of 8 dimensions
    const int r0 = lane >> 2, c0 = (lane & 3) * 2;
    float st[NT][4];
    float* Sg = S_state + (((size_t)slot * heads + h) * DIM + dq * (DIM / 4)) * vdim + p0 + grp * 16;
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[j][e] = Sg[(size_t)(j * 8 + c0 + (e & 1)) * vdim + r0 + (e >> 1) * 8];
    fetch(0);
    keep(0);
    for (int c = 0; c < nb; ++c) {
        const float decay = next_decay;
        if (c + 1 < nb) { fetch(c + 1); ask(c + 1); cp_async_wait<1>(); }
        else cp_async_wait<0>();
        __syncthreads();
        const uint32_t qb = smem_addr(raw_sm + (c & 1) * Z::BUF), kb = qb + Z::QK, vb = kb + Z::QK, pb = vb + Z::V;
        const float* te = tok + (c & 1) * 2 * CB;
        const float* tw = te + CB;
        float o[4][2][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
        // Q S over this warp's dimensions
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            uint32_t b0[2][3], b1[2][3];
            split3(st[2 * ks][0], st[2 * ks][1], b0[0]);
            split3(st[2 * ks + 1][0], st[2 * ks + 1][1], b1[0]);
            split3(st[2 * ks][2], st[2 * ks][3], b0[1]);
            split3(st[2 * ks + 1][2], st[2 * ks + 1][3], b1[1]);
            uint32_t a[4][4];
#pragma unroll
            for (int mt = 0; mt < 4; ++mt)
                ldmatrix_x4(tile_addr<DIM>(qb, mt * 16 + (lane & 15), (dq * KS + ks) * 2 + (lane >> 4)), a[mt][0], a[mt][1], a[mt][2], a[mt][3]);
#pragma unroll
            for (int i = 2; i >= 0; --i)                                   // the small parts first; eight sums side by side
#pragma unroll
                for (int mt = 0; mt < 4; ++mt) {
                    mma_bf16(o[mt][0], a[mt], b0[0][i], b1[0][i]);
                    mma_bf16(o[mt][1], a[mt], b0[1][i], b1[1][i]);
                }
        }
        // times e^(c_t), plus the block's own tokens: this warp's sixteen
        uint32_t vv[4];
        ldmatrix_x4_trans(v_addr(vb, dq * 16 + (lane & 15), grp * 2 + (lane >> 4)), vv[0], vv[1], vv[2], vv[3]);
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
            const float e0 = te[mt * 16 + r0], e1 = te[mt * 16 + r0 + 8];
#pragma unroll
            for (int j = 0; j < 2; ++j) { o[mt][j][0] *= e0; o[mt][j][1] *= e0; o[mt][j][2] *= e1; o[mt][j][3] *= e1; }
        }
#pragma unroll
        for (int i = 2; i >= 0; --i)
#pragma unroll
            for (int mt = 0; mt < 4; ++mt) {
                if (mt < dq) continue;                                     // tokens before this warp's
                uint32_t a[4];
                ldmatrix_x4(tile_addr<CB>(pb + i * PLANE * 2, mt * 16 + (lane & 15), dq * 2 + (lane >> 4)), a[0], a[1], a[2], a[3]);
                mma_bf16(o[mt][0], a, vv[0], vv[1]);
                mma_bf16(o[mt][1], a, vv[2], vv[3]);
            }
#pragma unroll
        for (int mt = 0; mt < 4; ++mt) {
            float* dst = red + ((size_t)dq * CB + mt * 16 + r0) * RED_LD + grp * 16 + c0;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                *reinterpret_cast<float2*>(dst + j * 8) = make_float2(o[mt][j][0], o[mt][j][1]);
                *reinterpret_cast<float2*>(dst + j * 8 + 8 * RED_LD) = make_float2(o[mt][j][2], o[mt][j][3]);
            }
        }
        // the state after the block
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) st[j][e] *= decay;
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
            uint32_t vr[4], a[3][4];
            ldmatrix_x4_trans(v_addr(vb, kt * 16 + (lane & 7) + ((lane >> 4) & 1) * 8, grp * 2 + ((lane >> 3) & 1)), vr[0], vr[1], vr[2], vr[3]);
            const float2 wa = *reinterpret_cast<const float2*>(tw + kt * 16 + c0), wb = *reinterpret_cast<const float2*>(tw + kt * 16 + 8 + c0);
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const float2 w = r < 2 ? wa : wb;
                uint32_t p[3];
                split3(__uint_as_float(vr[r] << 16) * w.x, __uint_as_float(vr[r] & 0xFFFF0000u) * w.y, p);
#pragma unroll
                for (int i = 0; i < 3; ++i) a[i][r] = p[i];
            }
            uint32_t kk[NT / 2][4];
#pragma unroll
            for (int j = 0; j < NT / 2; ++j)
                ldmatrix_x4_trans(tile_addr<DIM>(kb, kt * 16 + (lane & 15), dq * KS * 2 + 2 * j + (lane >> 4)), kk[j][0], kk[j][1], kk[j][2], kk[j][3]);
#pragma unroll
            for (int i = 2; i >= 0; --i)
#pragma unroll
                for (int j = 0; j < NT / 2; ++j) {
                    mma_bf16(st[2 * j], a[i], kk[j][0], kk[j][1]);
                    mma_bf16(st[2 * j + 1], a[i], kk[j][2], kk[j][3]);
                }
        }
        if (c + 1 < nb) keep(c + 1);              // (this place was last read before the block's first barrier)
        __syncthreads();                          // every part of the result is there, every tile has been read
        const int t0 = t_begin + c * CB, m = min(CB, n_tok - c * CB);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = (tid >> 3) + 32 * u, col = (tid & 7) * 4;
            if (r < m) {
                float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    float p[4];
                    load4(red + ((size_t)q * CB + r) * RED_LD + col, p);
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[e] += p[e];
                }
                store4(out + (size_t)(t0 + r) * ld_out + (size_t)h * vdim + p0 + col, v);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) Sg[(size_t)(j * 8 + c0 + (e & 1)) * vdim + r0 + (e >> 1) * 8] = st[j][e];
}
}  // namespace

// gates: float32 partial sums [n_in][T][row_stride]; log_keep, log_add, em: float32 [heads][T].
extern "C" int rb_mlstm_gates(const float* gates, int n_in, long long in_stride, int row_stride, int i_off, int f_off, float cap,
                              int heads, float* m_state, const int* seq_slot, const int* cu_q, const int* positions, int n_seqs,
                              int max_q_len, int T, float* log_keep, float* log_add, float* em, void* stream) {
    if (n_seqs <= 0 || T <= 0) return RB_OK;
    if (heads <= 0 || n_in < 1 || !(cap > 0.f) || n_seqs > 65535) return RB_ERR_BAD_SIZE;
    int threads = (max_q_len + 31) & ~31;
    threads = threads > 1024 ? 1024 : (threads < 32 ? 32 : threads);
    RB_LAUNCH((mlstm_gates_kernel), dim3(heads, n_seqs), dim3(threads), 0, (cudaStream_t)stream,
              Cols<float>{gates, n_in, (size_t)in_stride, row_stride}, i_off, f_off, cap, heads, m_state, seq_slot, cu_q, positions, T,
              log_keep, log_add, em);
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_mlstm_step(const void* x, int x_dtype, int n_in, long long in_stride, int row_stride, int q_off, int k_off, int v_off,
                             const float* gates, int g_n_in, long long g_in_stride, int g_row_stride, int i_off, int f_off, float cap,
                             float q_scale, float eps, int heads, int dim, int vdim, float* S_state, float* n_state, float* m_state,
                             const int* seq_slot, const int* cu_q, const int* positions, int n_seqs, float* out, int ld_out, float* den,
                             void* stream) {
    if (n_seqs <= 0) return RB_OK;
    if (heads <= 0 || dim <= 0 || vdim <= 0 || n_in < 1 || g_n_in < 1 || !(cap > 0.f) || n_seqs > 65535 || heads > 65535 || dim > 4096)
        return RB_ERR_BAD_SIZE;
    const dim3 grid((vdim + 31) / 32 + 1, heads, n_seqs);
    const size_t smem = (size_t)2 * dim * sizeof(float);
    const Cols<float> g{gates, g_n_in, (size_t)g_in_stride, g_row_stride};
#define RB_MS(IT)                                                                                                             \
    do {                                                                                                                      \
        const Cols<IT> c{(const IT*)x, n_in, (size_t)in_stride, row_stride};                                                  \
        if (vdim % 4 == 0 && !((uintptr_t)S_state & 15))                                                                      \
            RB_LAUNCH((mlstm_step_kernel<IT, 4>), grid, dim3(256), smem, (cudaStream_t)stream, c, q_off, k_off, v_off, g, i_off, f_off, \
                      cap, q_scale, eps, heads, dim, vdim, S_state, n_state, m_state, seq_slot, cu_q, positions, out, ld_out, den); \
        else                                                                                                                  \
            RB_LAUNCH((mlstm_step_kernel<IT, 1>), grid, dim3(256), smem, (cudaStream_t)stream, c, q_off, k_off, v_off, g, i_off, f_off, \
                      cap, q_scale, eps, heads, dim, vdim, S_state, n_state, m_state, seq_slot, cu_q, positions, out, ld_out, den); \
    } while (0)
    if (x_dtype == RB_F32) RB_MS(float);
    else if (x_dtype == RB_BF16) RB_MS(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_MS
    RB_LAUNCH_CHECK();
    return RB_OK;
}

// Prompts.  blocks >= the sum over the sequences of ceil(tokens / 64); work float32 [blocks][heads][dim][vdim], work_n
// [blocks][heads][dim], block_decay [blocks][heads], scores [blocks][heads][64][64]; out [T][heads * vdim], den [T][heads].
extern "C" int rb_mlstm_blocks(const void* x, int x_dtype, int n_in, long long in_stride, int row_stride, int q_off, int k_off, int v_off,
                               float q_scale, float eps, int heads, int dim, int vdim, const float* log_keep, const float* log_add,
                               const float* em, int T, float* S_state, float* n_state, const int* seq_slot, const int* cu_q, int n_seqs,
                               int blocks, float* work, float* work_n, float* block_decay, float* scores, float* out, int ld_out,
                               float* den, void* stream) {
    if (n_seqs <= 0 || blocks <= 0) return RB_OK;
    if (heads <= 0 || dim <= 0 || vdim <= 0 || n_in < 1 || n_seqs > 65535 || heads > 65535 || blocks > 65535) return RB_ERR_BAD_SIZE;
    cudaStream_t s = (cudaStream_t)stream;
    const dim3 grid((vdim + CB - 1) / CB, heads, blocks);
#define RB_MB(IT)                                                                                                             \
    do {                                                                                                                      \
        const Cols<IT> c{(const IT*)x, n_in, (size_t)in_stride, row_stride};                                                  \
        RB_LAUNCH((mlstm_block_scores_kernel<IT>), dim3(heads, blocks), dim3(CT), 0, s, c, q_off, k_off, q_scale, heads, dim, \
                  log_keep, log_add, T, seq_slot, cu_q, n_seqs, scores, den);                                                 \
        RB_LAUNCH((mlstm_block_sum_kernel<IT>), grid, dim3(CT), 0, s, c, k_off, v_off, heads, dim, vdim, log_keep, log_add, T, \
                  seq_slot, cu_q, n_seqs, work, work_n, block_decay);                                                         \
        RB_LAUNCH((mlstm_block_states_kernel), dim3((dim * vdim + dim + 255) / 256, heads, n_seqs), dim3(256), 0, s, work, work_n, \
                  block_decay, S_state, n_state, heads, dim, vdim, seq_slot, cu_q);                                           \
        RB_LAUNCH((mlstm_block_out_kernel<IT>), grid, dim3(CT), 0, s, c, q_off, v_off, q_scale, eps, heads, dim, vdim, log_keep, \
                  log_add, em, T, seq_slot, cu_q, n_seqs, work, work_n, scores, out, ld_out, den);                            \
    } while (0)
    if (x_dtype == RB_F32) RB_MB(float);
    else if (x_dtype == RB_BF16) RB_MB(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_MB
    RB_LAUNCH_CHECK();
    return RB_OK;
}

// The same for bfloat16 projection rows on the tensor cores: dim 64, 128, 192 or 256, vdim a multiple of 32, every head of q, k and v
// on a 16-byte boundary.  planes: bfloat16 [blocks][heads][3][64][64]; ec, wt: float32 [heads][T]; block_decay float32 [blocks][heads].
extern "C" int rb_mlstm_chain(const void* x, int row_stride, int q_off, int k_off, int v_off, float q_scale, float eps, int heads, int dim,
                              int vdim, const float* log_keep, const float* log_add, const float* em, int T, float* S_state, float* n_state,
                              const int* seq_slot, const int* cu_q, int n_seqs, int blocks, void* planes, float* ec, float* wt,
                              float* block_decay, float* out, int ld_out, float* den, void* stream) {
    if (n_seqs <= 0 || blocks <= 0) return RB_OK;
    if (heads <= 0 || vdim <= 0 || vdim % CHAIN_COLS || dim % 64 || dim < 64 || dim > 256 || n_seqs > 65535 || heads > 65535 || blocks > 65535)
        return RB_ERR_BAD_SIZE;
    if (((uintptr_t)x & 15) || row_stride % 8 || q_off % 8 || k_off % 8 || v_off % 8 || ((uintptr_t)planes & 15) || ((uintptr_t)out & 15) || ld_out % 4)
        return RB_ERR_BAD_ALIGN;
    cudaStream_t s = (cudaStream_t)stream;
    const Rows16 r{(const bf16*)x, row_stride};
    const dim3 grid(vdim / CHAIN_COLS + 1, heads, n_seqs);
#define RB_MC(DIM)                                                                                                                  \
    do {                                                                                                                            \
        auto k1 = mlstm_scores_tc_kernel<DIM>;                                                                                      \
        auto k2 = mlstm_chain_kernel<DIM>;                                                                                          \
        constexpr int sm1 = 2 * CB * DIM * 2, sm2 = ChainSizes<DIM>::SMEM;                                                          \
        cudaError_t e = cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, sm1);                                 \
        if (e == cudaSuccess) e = cudaFuncSetAttribute(k2, cudaFuncAttributeMaxDynamicSharedMemorySize, sm2);                       \
        if (e != cudaSuccess) return (int)e;                                                                                        \
        RB_LAUNCH((k1), dim3(heads, blocks), dim3(128), sm1, s, r, q_off, k_off, q_scale, heads, log_keep, log_add, T, seq_slot,    \
                  cu_q, n_seqs, (bf16*)planes, ec, wt, block_decay, den);                                                           \
        RB_LAUNCH((k2), grid, dim3(256), sm2, s, r, q_off, k_off, v_off, eps, heads, vdim, (const bf16*)planes, ec, wt, block_decay, \
                  em, T, S_state, n_state, seq_slot, cu_q, out, ld_out, den);                                                       \
    } while (0)
    if (dim == 64) RB_MC(64);
    else if (dim == 128) RB_MC(128);
    else if (dim == 192) RB_MC(192);
    else RB_MC(256);
#undef RB_MC
    RB_LAUNCH_CHECK();
    return RB_OK;
}
