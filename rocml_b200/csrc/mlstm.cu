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
// All arithmetic is 32-bit.  q, k, v are columns of the layer's projection, in the activations' type or as 32-bit partial
// sums that are added first; the gates' columns are 32-bit always.
#include "common.cuh"
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
        const IT* x = p + (size_t)t * row_stride + col;
        float v = 0.f;
        for (int s = 0; s < n_in; ++s) v += to_f32(x[(size_t)s * in_stride]);
        return v;
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
template <typename IT>
__global__ void __launch_bounds__(256)
mlstm_step_kernel(const Cols<IT> x, int q_off, int k_off, int v_off, const Cols<float> g, int i_off, int f_off, float cap,
                  float q_scale, float eps, int heads, int dim, int vdim, float* __restrict__ S_state, float* __restrict__ n_state,
                  float* __restrict__ m_state, const int* __restrict__ seq_slot, const int* __restrict__ cu_q,
                  const int* __restrict__ positions, float* __restrict__ out, int ld_out, float* __restrict__ den) {
    pdl_trigger();
    pdl_wait();
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
    const int pos = positions[t];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* mine = m_state + ((size_t)slot * heads + h) * 2;
    const float i = capped_gate(g(t, i_off + h), cap), f = log_sigmoid(capped_gate(g(t, f_off + h), cap));
    const float m0 = mine[(pos + 1) & 1], m1 = fmaxf(f + m0, i);
    const float keep = expf(f + m0 - m1), add = expf(i - m1);
    for (int c = threadIdx.x; c < dim; c += 256) {
        qs[c] = x(t, q_off + h * dim + c) * q_scale;
        ks[c] = x(t, k_off + h * dim + c) * add;
    }
    const bool last = blockIdx.x == gridDim.x - 1;          // this block does n, the divisor and m
    const int j = blockIdx.x * 32 + lane;
    float v = 0.f;
    if (!last && j < vdim) v = x(t, v_off + h * vdim + j);
    __syncthreads();
    if (last) {
        float* n = n_state + ((size_t)slot * heads + h) * dim;
        float acc = 0.f;
        for (int c = threadIdx.x; c < dim; c += 256) {
            const float s = fmaf(keep, n[c], ks[c]);
            n[c] = s;
            acc = fmaf(s, qs[c], acc);
        }
        acc = block_sum(acc, red);
        if (threadIdx.x == 0) {
            den[(size_t)t * heads + h] = fmaxf(fabsf(acc), expf(-m1)) + eps;
            mine[pos & 1] = m1;
        }
        return;
    }
    float* S = S_state + (((size_t)slot * heads + h) * dim) * vdim + j;
    float acc = 0.f;
    if (j < vdim) {
        int c = warp;
        for (; c + 56 < dim; c += 64) {           // eight rows' loads in flight
            float s[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) s[u] = S[(size_t)(c + 8 * u) * vdim];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                s[u] = fmaf(ks[c + 8 * u], v, keep * s[u]);
                S[(size_t)(c + 8 * u) * vdim] = s[u];
                acc = fmaf(s[u], qs[c + 8 * u], acc);
            }
        }
        for (; c < dim; c += 8) {
            const float s = fmaf(ks[c], v, keep * S[(size_t)c * vdim]);
            S[(size_t)c * vdim] = s;
            acc = fmaf(s, qs[c], acc);
        }
    }
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && j < vdim) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w][lane];
        out[(size_t)t * ld_out + (size_t)h * vdim + j] = o;
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
    RB_LAUNCH((mlstm_step_kernel<IT>), grid, dim3(256), smem, (cudaStream_t)stream,                                           \
              Cols<IT>{(const IT*)x, n_in, (size_t)in_stride, row_stride}, q_off, k_off, v_off, g, i_off, f_off, cap, q_scale, eps, \
              heads, dim, vdim, S_state, n_state, m_state, seq_slot, cu_q, positions, out, ld_out, den)
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
