// A real-gated linear recurrent unit: one state number a channel, decayed and fed by gates that each channel reads from its
// own block of channels.
//
//   r = sigmoid(Ra u + ba),  i = sigmoid(Ri u + bi)         block-diagonal: `blocks` square matrices [out, in] of `part`
//   log a = rate * r                                        rate [width] <= 0 (a negative constant times softplus of a weight)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u
//   out = S * gelu_tanh(y) * factor
//
//   rglru_gates   prompts: both block products of a tile of 64 tokens and 64 channels side by side, and from them the decay a
//                 and the input sqrt(1 - a^2) i u of every token and channel, next to each other.  With bfloat16 weights on the tensor
//                 cores (mma.sync): the 32-bit u enters as the sum of three bfloat16 numbers (24 bits), the sums are 32-bit, so
//                 the products are those of the 32-bit numbers.  Otherwise FMA.
//   rglru_scan    prompts: a block owns 16 channels of a sequence, half a warp one run of its tokens.  Each first forms its
//                 run's own sum and product of decays, then every half warp knows the state its run starts from, and walks it
//                 again to write the results.
//   rglru_step    one token a sequence: products, gates, recurrence and result in one kernel.
//
// Everything is 32-bit; u comes from the convolution in 32-bit, y is a column block of the projection.
#include "common.cuh"
#include "mma_tiles.cuh"
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
                   int T, float2* __restrict__ ax, int width) {
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
            ax[(size_t)t * width + ch] = make_float2(a, x);
        }
    }
}

// The same on the tensor cores.  A warp owns 16 tokens and 32 channels of both gates; a step of 64 inputs is split into its three
// planes as it is staged.
__global__ void __launch_bounds__(256)
rglru_gates_tc_kernel(const float* __restrict__ u, int ld_u, const __nv_bfloat16* __restrict__ ra, const __nv_bfloat16* __restrict__ ri,
                      const float* __restrict__ ra_b, const float* __restrict__ ri_b, const float* __restrict__ rate, int part, int tiles,
                      int T, float2* __restrict__ ax, int width) {
    using namespace mma_tiles;
    typedef __nv_bfloat16 bf16;
    pdl_trigger();
    pdl_wait();
    __shared__ __align__(128) bf16 Us[3][64 * 64], Rs[64 * 64], Is[64 * 64];       // rows of 64 inputs, swizzled
    const int blk = blockIdx.x / tiles, n0 = (blockIdx.x % tiles) * 64, m0 = blockIdx.y * 64;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int mt = warp & 3, nh = warp >> 2;
    const float* ub = u + (size_t)blk * part;
    const bf16* rw = ra + (size_t)blk * part * part;
    const bf16* iw = ri + (size_t)blk * part * part;
    float ar[4][4], ai[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) ar[j][e] = ai[j][e] = 0.f;
    const uint32_t u0 = smem_addr(Us[0]), rs = smem_addr(Rs), is = smem_addr(Is);
    for (int k0 = 0; k0 < part; k0 += 64) {
        __syncthreads();
#pragma unroll
        for (int v = 0; v < 2; ++v) {                                    // weights: 64 rows of eight 16-byte chunks each
            const int idx = tid + v * 256, r = idx >> 3, ch = idx & 7;
            const bool in = n0 + r < part && k0 + ch * 8 < part;
            const size_t at = in ? (size_t)(n0 + r) * part + k0 + ch * 8 : 0;
            cp_async16(reinterpret_cast<uint8_t*>(Rs) + r * 128 + ((ch ^ (r & 7)) << 4), rw + at, in);
            cp_async16(reinterpret_cast<uint8_t*>(Is) + r * 128 + ((ch ^ (r & 7)) << 4), iw + at, in);
        }
        cp_async_commit();
#pragma unroll
        for (int v = 0; v < 4; ++v) {                                    // inputs: four numbers a thread and turn
            const int idx = tid + v * 256, r = idx >> 4, c = (idx & 15) * 4;
            float f[4] = {0.f, 0.f, 0.f, 0.f};
            if (m0 + r < T && k0 + c < part) load4(ub + (size_t)(m0 + r) * ld_u + k0 + c, f);
            const int at = r * 128 + (((c >> 3) ^ (r & 7)) << 4) + (c & 4) * 2;
#pragma unroll
            for (int i = 0; i < 3; ++i) {
                const __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
                *reinterpret_cast<uint2*>(reinterpret_cast<uint8_t*>(Us[i]) + at) =
                    make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
                const float2 fa = __bfloat1622float2(a), fb = __bfloat1622float2(b);
                f[0] -= fa.x; f[1] -= fa.y; f[2] -= fb.x; f[3] -= fb.y;
            }
        }
        cp_async_wait<0>();
        __syncthreads();
        const int steps = min(4, (part - k0 + 15) / 16);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            if (ks >= steps) break;
            uint32_t a[3][4];
#pragma unroll
            for (int i = 0; i < 3; ++i)
                ldmatrix_x4(tile_addr<64>(u0 + i * 64 * 64 * 2, mt * 16 + (lane & 15), ks * 2 + (lane >> 4)), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int row = nh * 32 + j * 8 + (lane & 7) + ((lane >> 4) & 1) * 8, ch = ks * 2 + ((lane >> 3) & 1);
                uint32_t r0, r1, r2, r3, i0, i1, i2, i3;
                ldmatrix_x4(tile_addr<64>(rs, row, ch), r0, r1, r2, r3);
                ldmatrix_x4(tile_addr<64>(is, row, ch), i0, i1, i2, i3);
#pragma unroll
                for (int i = 2; i >= 0; --i) {                            // the small parts first
                    mma_bf16(ar[j], a[i], r0, r1);
                    mma_bf16(ar[j + 1], a[i], r2, r3);
                    mma_bf16(ai[j], a[i], i0, i1);
                    mma_bf16(ai[j + 1], a[i], i2, i3);
                }
            }
        }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int c = n0 + nh * 32 + j * 8 + (lane & 3) * 2;
        if (c >= part) continue;                                         // (part is even: both channels of a pair or none)
        const int ch = blk * part + c;
        const float2 rb = *reinterpret_cast<const float2*>(ra_b + ch), ib = *reinterpret_cast<const float2*>(ri_b + ch),
                     rt = *reinterpret_cast<const float2*>(rate + ch);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = m0 + mt * 16 + (lane >> 2) + 8 * e;
            if (t >= T) continue;
            const float2 uu = *reinterpret_cast<const float2*>(u + (size_t)t * ld_u + ch);
            float4 o;
            gate_pair(ar[j][2 * e] + rb.x, ai[j][2 * e] + ib.x, rt.x, uu.x, &o.x, &o.y);
            gate_pair(ar[j][2 * e + 1] + rb.y, ai[j][2 * e + 1] + ib.y, rt.y, uu.y, &o.z, &o.w);
            *reinterpret_cast<float4*>(ax + (size_t)t * width + ch) = o;
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
        const YT* x = p + (size_t)t * row_stride + c;
        float v = to_f32(x[0]);
        for (int s = 1; s < n_in; s += 4) {                 // four in flight, added in order
            float y[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = s + j < n_in ? to_f32(x[(size_t)(s + j) * in_stride]) : 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) v += y[j];
        }
        return v;
    }
};

constexpr int SCH = 16;            // channels a block
constexpr int SW = 32;             // runs of tokens: half a warp each (512 threads: several blocks a multiprocessor)
template <typename YT, typename AT>
__global__ void __launch_bounds__(SW * SCH)
rglru_scan_kernel(const float2* __restrict__ ax, int width, const Branch<YT> y, float factor, float* __restrict__ state,
                  const int* __restrict__ seq_slot, const int* __restrict__ cu_q, AT* __restrict__ out, int ld_out) {
    pdl_wait();                                     // (no early signal: few blocks that run long)
    __shared__ float prod[SW][SCH], own[SW][SCH];
    const int b = blockIdx.y;
    const int slot = seq_slot[b];
    if (slot < 0) return;
    const int t0 = cu_q[b], n = cu_q[b + 1] - t0;
    if (n <= 0) return;
    const int run = threadIdx.x / SCH, lane = threadIdx.x % SCH;
    const int c = blockIdx.x * SCH + lane;
    const bool here = c < width;
    const int len = (n + SW - 1) / SW;
    const int lo = min(n, run * len), hi = min(n, lo + len);
    const float2* p = ax + (size_t)t0 * width + c;
    float* st = state + (size_t)slot * width + c;
    const float start = here ? *st : 0.f;           // every run reads it before the barrier, one writes it after
    float P = 1.f, S = 0.f;
    constexpr int U = 16;
    if (here) {
        for (int t = lo; t < hi; t += U) {
            float2 v[U];
#pragma unroll
            for (int j = 0; j < U; ++j) v[j] = t + j < hi ? p[(size_t)(t + j) * width] : make_float2(1.f, 0.f);
#pragma unroll
            for (int j = 0; j < U; ++j) { S = fmaf(v[j].x, S, v[j].y); P *= v[j].x; }
        }
    }
    prod[run][lane] = P;
    own[run][lane] = S;
    __syncthreads();
    if (!here || lo >= hi) return;
    S = start;
    for (int w = 0; w < run; ++w) S = fmaf(prod[w][lane], S, own[w][lane]);
    AT* op = out + (size_t)t0 * ld_out + c;
    constexpr int U2 = 8;
    for (int t = lo; t < hi; t += U2) {
        float2 v[U2];
        float yv[U2];
#pragma unroll
        for (int j = 0; j < U2; ++j) {
            v[j] = t + j < hi ? p[(size_t)(t + j) * width] : make_float2(1.f, 0.f);
            yv[j] = t + j < hi ? y(t0 + t + j, c) : 0.f;
        }
#pragma unroll
        for (int j = 0; j < U2; ++j) {
            S = fmaf(v[j].x, S, v[j].y);
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
    // what this lane will end up with: its state and its part of the other branch are asked for before the products
    const int r0 = n0 + warp * 4;
    const int c = r0 + (lane >> 3), t = t0 + (lane & 7), ch = blk * part + c;
    const bool mine = c < part && t < T;
    const int slot = mine ? slot_of_token[t] : -1;
    float* st = state + (size_t)(slot < 0 ? 0 : slot) * width + (mine ? ch : 0);
    float before = 0.f, yv = 0.f, zr = 0.f, zi = 0.f, rt = 0.f;
    if (slot >= 0) { before = *st; yv = y(t, ch); zr = ra_b[ch]; zi = ri_b[ch]; rt = rate[ch]; }
    __syncthreads();
    float v[64];
#pragma unroll
    for (int j = 0; j < 64; ++j) v[j] = 0.f;
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
    if (slot < 0) return;
    float a, x;
    gate_pair(v[0] + zr, v[1] + zi, rt, us[(lane & 7) * part + c], &a, &x);
    const float S = fmaf(a, before, x);
    *st = S;
    out[(size_t)t * ld_out + ch] = from_f32<AT>(S * gelu_tanh(yv) * factor);
}
}  // namespace

extern "C" int rb_rglru_gates(const float* u, int ld_u, const void* ra, const void* ri, int w_dtype, const float* ra_b, const float* ri_b,
                              const float* rate, int blocks, int part, int T, float* ax, void* stream) {
    if (T <= 0) return RB_OK;
    if (blocks <= 0 || part <= 0) return RB_ERR_BAD_SIZE;
    const int tiles = (part + TN - 1) / TN;
    const dim3 grid(blocks * tiles, (T + TM - 1) / TM);
    if (grid.y > 65535) return RB_ERR_BAD_SIZE;
    if (w_dtype == RB_BF16 && part % 8 == 0 && ld_u % 4 == 0 && (((uintptr_t)u | (uintptr_t)ra | (uintptr_t)ri | (uintptr_t)ax) & 15) == 0 &&
        (((uintptr_t)ra_b | (uintptr_t)ri_b | (uintptr_t)rate) & 7) == 0) {
        RB_LAUNCH((rglru_gates_tc_kernel), grid, dim3(256), 0, (cudaStream_t)stream, u, ld_u, (const __nv_bfloat16*)ra, (const __nv_bfloat16*)ri,
                  ra_b, ri_b, rate, part, tiles, T, (float2*)ax, blocks * part);
        RB_LAUNCH_CHECK();
        return RB_OK;
    }
#define RB_RG(WT)                                                                                                               \
    RB_LAUNCH((rglru_gates_kernel<WT>), grid, dim3(256), 0, (cudaStream_t)stream, u, ld_u, (const WT*)ra, (const WT*)ri, ra_b,  \
              ri_b, rate, part, tiles, T, (float2*)ax, blocks * part)
    if (w_dtype == RB_F32) RB_RG(float);
    else if (w_dtype == RB_BF16) RB_RG(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_RG
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_rglru_scan(const float* ax, int width, const void* y, int y_dtype, int n_in, long long in_stride,
                             int row_stride, float factor, float* state, const int* seq_slot, const int* cu_q, int n_seqs, void* out,
                             int out_dtype, int ld_out, void* stream) {
    if (n_seqs <= 0) return RB_OK;
    if (width <= 0 || n_in < 1 || n_seqs > 65535) return RB_ERR_BAD_SIZE;
    if ((uintptr_t)ax & 7) return RB_ERR_BAD_ALIGN;
    const dim3 grid((width + SCH - 1) / SCH, n_seqs);
    typedef __nv_bfloat16 bf;
#define RB_RS(YT, AT)                                                                                                            \
    RB_LAUNCH((rglru_scan_kernel<YT, AT>), grid, dim3(SW * SCH), 0, (cudaStream_t)stream, (const float2*)ax, width,                            \
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
