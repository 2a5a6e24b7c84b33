// A real-gated linear recurrent unit: one state number a channel, decayed and fed by gates that each channel reads from its
// own block of channels.
//
//   r = sigmoid(Ra u + ba),  i = sigmoid(Ri u + bi)         block-diagonal: `blocks` square matrices [out, in] of `part`
//   log a = rate * r                                        rate [width] <= 0 (a negative constant times softplus of a weight)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u
//   out = S * gelu_tanh(y) * factor
//
//   rglru_gates   prompts: both block products of a tile of 64 tokens and 64 channels side by side, and from them the decay a
//                 and the input sqrt(1 - a^2) i u of every token and channel.
//   rglru_scan    prompts: a block owns 32 channels of a sequence, a warp one run of its tokens.  Each warp first forms its
//                 run's own sum and product of decays, then every warp knows the state its run starts from, and walks it
//                 again to write the results.
//   rglru_step    one token a sequence: products, gates, recurrence and result in one kernel.
//
// Everything is 32-bit; u comes from the convolution in 32-bit, y is a column block of the projection.
#include "common.cuh"
#include "api.h"

using namespace rb;

namespace {
constexpr int TM = 64, TN = 64, TK = 32;      // tokens, channels and products' depth of a tile
constexpr int LD = TM + 4;

__device__ __forceinline__ void gate_pair(float zr, float zi, float rate, float u, float* a, float* x) {
    const float la = rate * sigmoid_f32(zr);
    *a = expf(la);
    *x = sqrtf(-expm1f(2.f * la)) * sigmoid_f32(zi) * u;
}

template <typename WT>
__global__ void __launch_bounds__(256)
rglru_gates_kernel(const float* __restrict__ u, int ld_u, const WT* __restrict__ ra, const WT* __restrict__ ri,
                   const float* __restrict__ ra_b, const float* __restrict__ ri_b, const float* __restrict__ rate, int part, int tiles,
                   int T, float* __restrict__ a_out, float* __restrict__ x_out, int width) {
    pdl_trigger();
    pdl_wait();
    __shared__ __align__(16) float Us[TK * LD], Rs[TK * LD], Is[TK * LD];
    const int blk = blockIdx.x / tiles, n0 = (blockIdx.x % tiles) * TN, m0 = blockIdx.y * TM;
    const int ty = threadIdx.x >> 4, tx = threadIdx.x & 15;
    const float* ub = u + (size_t)blk * part;
    const WT* rw = ra + (size_t)blk * part * part;
    const WT* iw = ri + (size_t)blk * part * part;
    float ar[4][4] = {}, ai[4][4] = {};
    for (int k0 = 0; k0 < part; k0 += TK) {
        __syncthreads();
        for (int idx = threadIdx.x; idx < TM * TK; idx += 256) {
            const int row = idx / TK, k = idx - row * TK;
            const bool kin = k0 + k < part;
            Us[k * LD + row] = kin && m0 + row < T ? ub[(size_t)(m0 + row) * ld_u + k0 + k] : 0.f;
            const bool win = kin && n0 + row < part;
            Rs[k * LD + row] = win ? to_f32(rw[(size_t)(n0 + row) * part + k0 + k]) : 0.f;
            Is[k * LD + row] = win ? to_f32(iw[(size_t)(n0 + row) * part + k0 + k]) : 0.f;
        }
        __syncthreads();
        const int kk = min(TK, part - k0);
#pragma unroll 4
        for (int k = 0; k < kk; ++k) {
            float a[4], r[4], i[4];
            load4(Us + k * LD + 4 * ty, a);
            load4(Rs + k * LD + 4 * tx, r);
            load4(Is + k * LD + 4 * tx, i);
#pragma unroll
            for (int p = 0; p < 4; ++p)
#pragma unroll
                for (int q = 0; q < 4; ++q) { ar[p][q] = fmaf(a[p], r[q], ar[p][q]); ai[p][q] = fmaf(a[p], i[q], ai[p][q]); }
        }
    }
#pragma unroll
    for (int p = 0; p < 4; ++p) {
        const int t = m0 + 4 * ty + p;
        if (t >= T) continue;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
            const int c = n0 + 4 * tx + q;
            if (c >= part) continue;
            const int ch = blk * part + c;
            float a, x;
            gate_pair(ar[p][q] + ra_b[ch], ai[p][q] + ri_b[ch], rate[ch], u[(size_t)t * ld_u + ch], &a, &x);
            a_out[(size_t)t * width + ch] = a;
            x_out[(size_t)t * width + ch] = x;
        }
    }
}

template <typename YT>
struct Branch {            // the other branch's columns of the projection rows: partial sums, added in order
    const YT* p;
    int n_in;
    size_t in_stride;
    int row_stride;
    __device__ __forceinline__ float operator()(int t, int c) const {
        float v = 0.f;
        for (int s = 0; s < n_in; ++s) v += to_f32(p[(size_t)s * in_stride + (size_t)t * row_stride + c]);
        return v;
    }
};

constexpr int SW = 32;             // warps a block: runs of tokens
template <typename YT, typename AT>
__global__ void __launch_bounds__(SW * 32)
rglru_scan_kernel(const float* __restrict__ a, const float* __restrict__ x, int width, const Branch<YT> y, float factor,
                  float* __restrict__ state, const int* __restrict__ seq_slot, const int* __restrict__ cu_q, AT* __restrict__ out, int ld_out) {
    pdl_trigger();
    pdl_wait();
    __shared__ float prod[SW][32], own[SW][32];
    const int b = blockIdx.y;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
    if (n <= 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x * 32 + lane;
    const bool here = c < width;
    const int run = (n + SW - 1) / SW;
    const int lo = min(n, warp * run), hi = min(n, lo + run);
    const float* ap = a + (size_t)t0 * width + c;
    const float* xp = x + (size_t)t0 * width + c;
    float* st = state + (size_t)slot * width + c;
    const float start = here ? *st : 0.f;           // every warp reads it before the barrier, one writes it after
    float P = 1.f, S = 0.f;
    constexpr int U = 8;
    if (here) {
        for (int t = lo; t < hi; t += U) {
            float av[U], xv[U];
#pragma unroll
            for (int j = 0; j < U; ++j) {
                av[j] = t + j < hi ? ap[(size_t)(t + j) * width] : 1.f;
                xv[j] = t + j < hi ? xp[(size_t)(t + j) * width] : 0.f;
            }
#pragma unroll
            for (int j = 0; j < U; ++j) { S = fmaf(av[j], S, xv[j]); P *= av[j]; }
        }
    }
    prod[warp][lane] = P;
    own[warp][lane] = S;
    __syncthreads();
    if (!here || lo >= hi) return;
    S = start;
    for (int w = 0; w < warp; ++w) S = fmaf(prod[w][lane], S, own[w][lane]);
    AT* op = out + (size_t)t0 * ld_out + c;
    for (int t = lo; t < hi; t += U) {
        float av[U], xv[U], yv[U];
#pragma unroll
        for (int j = 0; j < U; ++j) {
            av[j] = t + j < hi ? ap[(size_t)(t + j) * width] : 1.f;
            xv[j] = t + j < hi ? xp[(size_t)(t + j) * width] : 0.f;
            yv[j] = t + j < hi ? y(t0 + t + j, c) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < U; ++j) {
            S = fmaf(av[j], S, xv[j]);
            if (t + j < hi) op[(size_t)(t + j) * ld_out] = from_f32<AT>(S * gelu_tanh(yv[j]) * factor);
        }
    }
    if (hi == n) *st = S;
}

// One token a sequence: a block takes up to eight tokens and 32 channels, a warp four channels.  A lane's sixty-four sums (four
// channels, eight tokens, two gates) over its part of the block's inputs meet by halving exchanges, after which every lane
// holds both gates' sums of one (channel, token) and finishes it.
constexpr int ST = 8;
template <typename WT, typename YT, typename AT, int V>
__global__ void __launch_bounds__(256)
rglru_step_kernel(const float* __restrict__ u, int ld_u, const WT* __restrict__ ra, const WT* __restrict__ ri,
                  const float* __restrict__ ra_b, const float* __restrict__ ri_b, const float* __restrict__ rate, int part, int tiles,
                  int T, int width, const Branch<YT> y, float factor, float* __restrict__ state, const int* __restrict__ slot_of_token,
                  AT* __restrict__ out, int ld_out) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float us[];            // [ST][part]
    const int blk = blockIdx.x / tiles, n0 = (blockIdx.x % tiles) * 32, t0 = blockIdx.y * ST;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int idx = threadIdx.x; idx < ST * part; idx += 256) {
        const int t = idx / part, k = idx - t * part;
        us[idx] = t0 + t < T ? u[(size_t)(t0 + t) * ld_u + (size_t)blk * part + k] : 0.f;
    }
    __syncthreads();
    float v[64];
#pragma unroll
    for (int j = 0; j < 64; ++j) v[j] = 0.f;
    const int r0 = n0 + warp * 4;
    for (int k = lane * V; k < part; k += 32 * V) {
        float uv[ST][V];
#pragma unroll
        for (int t = 0; t < ST; ++t) {
            if (V == 4) load4(us + t * part + k, uv[t]);
            else uv[t][0] = us[t * part + k];
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            if (r0 + j >= part) continue;
            const size_t at = ((size_t)blk * part + r0 + j) * part + k;
            float wr[V], wi[V];
            if (V == 4) { load4(ra + at, wr); load4(ri + at, wi); }
            else { wr[0] = to_f32(ra[at]); wi[0] = to_f32(ri[at]); }
#pragma unroll
            for (int t = 0; t < ST; ++t)
#pragma unroll
                for (int q = 0; q < V; ++q) {
                    v[(j * ST + t) * 2] = fmaf(wr[q], uv[t][q], v[(j * ST + t) * 2]);
                    v[(j * ST + t) * 2 + 1] = fmaf(wi[q], uv[t][q], v[(j * ST + t) * 2 + 1]);
                }
        }
    }
#pragma unroll
    for (int o = 16, n = 32; o > 0; o >>= 1, n >>= 1)
#pragma unroll
        for (int j = 0; j < 32; ++j)
            if (j < n) {
                const bool up = (lane & o) != 0;
                const float mine = up ? v[j + n] : v[j], other = up ? v[j] : v[j + n];
                v[j] = mine + __shfl_xor_sync(0xffffffffu, other, o);
            }
    const int c = r0 + (lane >> 3), t = t0 + (lane & 7);        // what this lane ended up with
    if (c >= part || t >= T) return;
    const int slot = slot_of_token[t];
    if (slot < 0) return;
    const int ch = blk * part + c;
    float a, x;
    gate_pair(v[0] + ra_b[ch], v[1] + ri_b[ch], rate[ch], us[(lane & 7) * part + c], &a, &x);
    float* st = state + (size_t)slot * width + ch;
    const float S = fmaf(a, *st, x);
    *st = S;
    out[(size_t)t * ld_out + ch] = from_f32<AT>(S * gelu_tanh(y(t, ch)) * factor);
}
}  // namespace

extern "C" int rb_rglru_gates(const float* u, int ld_u, const void* ra, const void* ri, int w_dtype, const float* ra_b, const float* ri_b,
                              const float* rate, int blocks, int part, int T, float* a, float* x, void* stream) {
    if (T <= 0) return RB_OK;
    if (blocks <= 0 || part <= 0) return RB_ERR_BAD_SIZE;
    const int tiles = (part + TN - 1) / TN;
    const dim3 grid(blocks * tiles, (T + TM - 1) / TM);
    if (grid.y > 65535) return RB_ERR_BAD_SIZE;
#define RB_RG(WT)                                                                                                               \
    RB_LAUNCH((rglru_gates_kernel<WT>), grid, dim3(256), 0, (cudaStream_t)stream, u, ld_u, (const WT*)ra, (const WT*)ri, ra_b,  \
              ri_b, rate, part, tiles, T, a, x, blocks * part)
    if (w_dtype == RB_F32) RB_RG(float);
    else if (w_dtype == RB_BF16) RB_RG(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_RG
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_rglru_scan(const float* a, const float* x, int width, const void* y, int y_dtype, int n_in, long long in_stride,
                             int row_stride, float factor, float* state, const int* seq_slot, const int* cu_q, int n_seqs, void* out,
                             int out_dtype, int ld_out, void* stream) {
    if (n_seqs <= 0) return RB_OK;
    if (width <= 0 || n_in < 1 || n_seqs > 65535) return RB_ERR_BAD_SIZE;
    const dim3 grid((width + 31) / 32, n_seqs);
    typedef __nv_bfloat16 bf;
#define RB_RS(YT, AT)                                                                                                            \
    RB_LAUNCH((rglru_scan_kernel<YT, AT>), grid, dim3(SW * 32), 0, (cudaStream_t)stream, a, x, width,                            \
              Branch<YT>{(const YT*)y, n_in, (size_t)in_stride, row_stride}, factor, state, seq_slot, cu_q, (AT*)out, ld_out)
    if (y_dtype == RB_BF16 && out_dtype == RB_BF16) RB_RS(bf, bf);
    else if (y_dtype == RB_F32 && out_dtype == RB_BF16) RB_RS(float, bf);
    else if (y_dtype == RB_F32 && out_dtype == RB_F32) RB_RS(float, float);
    else return RB_ERR_BAD_DTYPE;
#undef RB_RS
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_rglru_step(const float* u, int ld_u, const void* ra, const void* ri, int w_dtype, const float* ra_b, const float* ri_b,
                             const float* rate, int blocks, int part, int T, const void* y, int y_dtype, int n_in, long long in_stride,
                             int row_stride, float factor, float* state, const int* slot_of_token, void* out, int out_dtype, int ld_out,
                             void* stream) {
    if (T <= 0) return RB_OK;
    if (blocks <= 0 || part <= 0 || n_in < 1) return RB_ERR_BAD_SIZE;
    const size_t smem = (size_t)ST * part * sizeof(float);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    const int tiles = (part + 31) / 32;
    const dim3 grid(blocks * tiles, (T + ST - 1) / ST);
    if (grid.y > 65535) return RB_ERR_BAD_SIZE;
    const size_t wsz = w_dtype == RB_F32 ? 4 : 2;
    const bool vec = part % 4 == 0 && (((uintptr_t)ra | (uintptr_t)ri) & (4 * wsz - 1)) == 0;
    typedef __nv_bfloat16 bf;
#define RB_RT(WT, YT, AT, V)                                                                                                      \
    do {                                                                                                                          \
        auto k = rglru_step_kernel<WT, YT, AT, V>;                                                                                \
        if (smem > 48 * 1024) {                                                                                                   \
            cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                      \
            if (e != cudaSuccess) return (int)e;                                                                                  \
        }                                                                                                                         \
        RB_LAUNCH((k), grid, dim3(256), smem, (cudaStream_t)stream, u, ld_u, (const WT*)ra, (const WT*)ri, ra_b, ri_b, rate, part, \
                  tiles, T, blocks * part, Branch<YT>{(const YT*)y, n_in, (size_t)in_stride, row_stride}, factor, state,          \
                  slot_of_token, (AT*)out, ld_out);                                                                               \
    } while (0)
#define RB_RV(WT, YT, AT) do { if (vec) RB_RT(WT, YT, AT, 4); else RB_RT(WT, YT, AT, 1); } while (0)
    if (w_dtype == RB_BF16 && y_dtype == RB_BF16 && out_dtype == RB_BF16) RB_RV(bf, bf, bf);
    else if (w_dtype == RB_BF16 && y_dtype == RB_F32 && out_dtype == RB_BF16) RB_RV(bf, float, bf);
    else if (w_dtype == RB_F32 && y_dtype == RB_F32 && out_dtype == RB_F32) RB_RV(float, float, float);
    else if (w_dtype == RB_F32 && y_dtype == RB_F32 && out_dtype == RB_BF16) RB_RV(float, float, bf);
    else if (w_dtype == RB_F32 && y_dtype == RB_BF16 && out_dtype == RB_BF16) RB_RV(float, bf, bf);
    else return RB_ERR_BAD_DTYPE;
#undef RB_RV
#undef RB_RT
    RB_LAUNCH_CHECK();
    return RB_OK;
}
