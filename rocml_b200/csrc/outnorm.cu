// Layer norms, and norms of a sublayer's result.
//
//   add_layernorm  r = resid[row] + sum of the partial sums; optionally written back; out = (r - mean) / sqrt(var + eps) * w + b
//                  with var the mean of the squared deviations.  The layer-norm twin of add_rmsnorm (elementwise.cu).
//   out_norm       resid[row] += mult * norm(d), in place; d = d_scale * (the sum of the sublayer's partial sums), or, for a routed
//                  feed-forward, d_scale * (sum_j weights[t, j] * delta[row_of[t, j]] + self_weight[t] * self_x[t]); norm is a
//                  layer norm or an RMS norm with a weight and an optional bias.  The new row is also written in the type
//                  of the product that reads it next, because the sublayers of such a layer read the stream itself.
//
//   pair_norm      the same for a sublayer with two results that are normalised apart and added: d = factor * (rms(a) * wa + rms(b) * wb).
//
// One block a row, the row in shared memory between the passes (mean, squared deviations, result), 16-byte accesses
// where width and addresses allow.  All arithmetic is 32-bit; partial sums are added in their order, so a row's result
// depends on nothing else in the batch.
#include "common.cuh"
#include "api.h"

using namespace rb;

namespace {
// (row - mean) statistics of `row` [H] in shared memory: mean (0 for an RMS norm) and 1 / sqrt(var + eps).  `sum` is this
// thread's part of the row's sum.
__device__ __forceinline__ void row_statistics(const float* row, int H, bool layer, float sum, float eps, float* red, float* mean,
                                               float* rstd) {
    const float mu = layer ? block_sum(sum, red) / (float)H : 0.f;
    if (!layer) __syncthreads();
    float ss = 0.f;
    if ((H & 3) == 0) {
        for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
            float v[4];
            load4(row + i, v);
#pragma unroll
            for (int u = 0; u < 4; ++u) ss = fmaf(v[u] - mu, v[u] - mu, ss);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) ss = fmaf(row[i] - mu, row[i] - mu, ss);
    }
    *rstd = rsqrtf(block_sum(ss, red) / (float)H + eps);
    *mean = mu;
}

template <typename OT>
__global__ void __launch_bounds__(1024)
add_layernorm_kernel(float* __restrict__ resid, const float* __restrict__ delta, int n_delta, size_t delta_stride,
                     const float* __restrict__ w, const float* __restrict__ b, OT* __restrict__ out, const int* __restrict__ rows,
                     int H, float eps, int write_back, int vec) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row[];       // H floats (padded to 4) + 33
    float* red = row + ((H + 3) & ~3);
    const int src = rows ? rows[blockIdx.x] : blockIdx.x;
    if (src < 0) return;                                // a padded entry
    float* x = resid + (size_t)src * H;
    const float* d = delta + (size_t)src * H;
    OT* o = out + (size_t)blockIdx.x * H;
    float sum = 0.f, mean, rstd;
    if (vec) {
        for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
            float v[4], p[4];
            load4(x + i, v);
            for (int s = 0; s < n_delta; ++s) {
                load4(d + (size_t)s * delta_stride + i, p);
#pragma unroll
                for (int u = 0; u < 4; ++u) v[u] += p[u];
            }
            sum += v[0] + v[1] + v[2] + v[3];
            store4(row + i, v);
            if (write_back) store4(x + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            float v = x[i];
            for (int s = 0; s < n_delta; ++s) v += d[(size_t)s * delta_stride + i];
            sum += v;
            row[i] = v;
            if (write_back) x[i] = v;
        }
    }
    row_statistics(row, H, true, sum, eps, red, &mean, &rstd);
    if (vec) {
        for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
            float v[4], ww[4], bb[4] = {0.f, 0.f, 0.f, 0.f};
            load4(row + i, v);
            load4(w + i, ww);
            if (b) load4(b + i, bb);
#pragma unroll
            for (int u = 0; u < 4; ++u) v[u] = fmaf((v[u] - mean) * rstd, ww[u], bb[u]);
            store4(o + i, v);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x)
            o[i] = from_f32<OT>(fmaf((row[i] - mean) * rstd, w[i], b ? b[i] : 0.f));
    }
}

struct Routed {
    const int* row_of;             // null: delta are partial sums
    const float* weights;
    int top;
    const float* self_weight;      // may be null
};

// Two results of one sublayer, each normalised on its own: v = factor * (rms(a) * wa + rms(b) * wb), a and b sums of partial sums.
// Without `w` v is the result (out_v float32 [T, H]); with it resid[row] += mult * rms(v) * w, and `out` receives the new row.
template <typename OT>
__global__ void __launch_bounds__(1024)
pair_norm_kernel(const float* __restrict__ da, int na, size_t sa, const float* __restrict__ db, int nb, size_t sb,
                 const float* __restrict__ wa, const float* __restrict__ wb, float eps_in, float factor, float* __restrict__ out_v,
                 float* __restrict__ resid, const float* __restrict__ w, float eps, float mult, OT* __restrict__ out, int H, int vec) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row[];       // 2 rows of H floats (padded to 4) + 2 * 33
    const int ldr = (H + 3) & ~3;
    float* row_b = row + ldr;
    float* red = row_b + ldr;
    const int t = blockIdx.x;
    float s0 = 0.f, s1 = 0.f;
    for (int part = 0; part < 2; ++part) {
        const float* d = (part ? db : da) + (size_t)t * H;
        const int nd = part ? nb : na;
        const size_t st = part ? sb : sa;
        float* dst = part ? row_b : row;
        float ss = 0.f;
        if (vec) {
            for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                for (int s = 0; s < nd; s += 4) {          // four partial sums in flight, added in order
                    float p[4][4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (s + j < nd) load4(d + (size_t)(s + j) * st + i, p[j]);
                        else p[j][0] = p[j][1] = p[j][2] = p[j][3] = 0.f;
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int u = 0; u < 4; ++u) v[u] += p[j][u];
                }
                ss += v[0] * v[0] + v[1] * v[1] + v[2] * v[2] + v[3] * v[3];
                store4(dst + i, v);
            }
        } else {
            for (int i = threadIdx.x; i < H; i += blockDim.x) {
                float v = 0.f;
                for (int s = 0; s < nd; ++s) v += d[(size_t)s * st + i];
                ss = fmaf(v, v, ss);
                dst[i] = v;
            }
        }
        if (part) s1 = ss; else s0 = ss;
    }
    s0 = block_sum(s0, red);
    s1 = block_sum(s1, red + 33);
    const float ia = rsqrtf(s0 / (float)H + eps_in) * factor, ib = rsqrtf(s1 / (float)H + eps_in) * factor;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = row[i] * ia * wa[i] + row_b[i] * ib * wb[i];
        row[i] = v;
        ss = fmaf(v, v, ss);
        if (!w) out_v[(size_t)t * H + i] = v;
    }
    if (!w) return;
    const float inv = rsqrtf(block_sum(ss, red) / (float)H + eps) * mult;
    float* x = resid + (size_t)t * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float v = fmaf(row[i] * inv, w[i], x[i]);
        x[i] = v;
        if (out) out[(size_t)t * H + i] = from_f32<OT>(v);
    }
}

template <typename OT, typename XT>
__global__ void __launch_bounds__(1024)
out_norm_kernel(float* __restrict__ resid, const float* __restrict__ delta, int n_delta, size_t delta_stride, float d_scale,
                const Routed routed, const XT* __restrict__ self_x, int layer, const float* __restrict__ w,
                const float* __restrict__ b, float eps, float mult, OT* __restrict__ out, int H, int vec) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row[];       // H floats (padded to 4) + 33
    float* red = row + ((H + 3) & ~3);
    const int t = blockIdx.x;
    float* x = resid + (size_t)t * H;
    float sum = 0.f, mean, rstd;
    if (routed.row_of) {
        const float sw = routed.self_weight ? routed.self_weight[t] : 0.f;
        const int* places = routed.row_of + (size_t)t * routed.top;
        const float* wt = routed.weights + (size_t)t * routed.top;
        if (vec) {
            for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
                float v[4] = {0.f, 0.f, 0.f, 0.f}, p[4];
                for (int j = 0; j < routed.top; ++j) {
                    const int src = places[j];
                    if (src < 0) continue;
                    const float f = wt[j];
                    load4(delta + (size_t)src * delta_stride + i, p);
#pragma unroll
                    for (int u = 0; u < 4; ++u) v[u] = fmaf(f, p[u], v[u]);
                }
                if (sw != 0.f) {
                    load4(self_x + (size_t)t * H + i, p);
#pragma unroll
                    for (int u = 0; u < 4; ++u) v[u] = fmaf(sw, p[u], v[u]);
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) v[u] *= d_scale;
                sum += v[0] + v[1] + v[2] + v[3];
                store4(row + i, v);
            }
        } else {
            for (int i = threadIdx.x; i < H; i += blockDim.x) {
                float v = 0.f;
                for (int j = 0; j < routed.top; ++j)
                    if (places[j] >= 0) v = fmaf(wt[j], delta[(size_t)places[j] * delta_stride + i], v);
                if (sw != 0.f) v = fmaf(sw, to_f32(self_x[(size_t)t * H + i]), v);
                v *= d_scale;
                sum += v;
                row[i] = v;
            }
        }
    } else {
        const float* d = delta + (size_t)t * H;
        if (vec) {
            for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
                float v[4] = {0.f, 0.f, 0.f, 0.f};
                for (int s = 0; s < n_delta; s += 4) {          // four partial sums in flight, added in order
                    float p[4][4];
#pragma unroll
                    for (int j = 0; j < 4; ++j) {
                        if (s + j < n_delta) load4(d + (size_t)(s + j) * delta_stride + i, p[j]);
                        else p[j][0] = p[j][1] = p[j][2] = p[j][3] = 0.f;
                    }
#pragma unroll
                    for (int j = 0; j < 4; ++j)
#pragma unroll
                        for (int u = 0; u < 4; ++u) v[u] += p[j][u];
                }
#pragma unroll
                for (int u = 0; u < 4; ++u) v[u] *= d_scale;
                sum += v[0] + v[1] + v[2] + v[3];
                store4(row + i, v);
            }
        } else {
            for (int i = threadIdx.x; i < H; i += blockDim.x) {
                float v = 0.f;
                for (int s = 0; s < n_delta; ++s) v += d[(size_t)s * delta_stride + i];
                v *= d_scale;
                sum += v;
                row[i] = v;
            }
        }
    }
    row_statistics(row, H, layer != 0, sum, eps, red, &mean, &rstd);
    if (vec) {
        for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
            float v[4], ww[4], bb[4] = {0.f, 0.f, 0.f, 0.f}, xx[4];
            load4(row + i, v);
            load4(w + i, ww);
            if (b) load4(b + i, bb);
            load4(x + i, xx);
#pragma unroll
            for (int u = 0; u < 4; ++u) xx[u] = fmaf(mult, fmaf((v[u] - mean) * rstd, ww[u], bb[u]), xx[u]);
            store4(x + i, xx);
            if (out) store4(out + (size_t)t * H + i, xx);
        }
    } else {
        for (int i = threadIdx.x; i < H; i += blockDim.x) {
            const float v = fmaf(mult, fmaf((row[i] - mean) * rstd, w[i], b ? b[i] : 0.f), x[i]);
            x[i] = v;
            if (out) out[(size_t)t * H + i] = from_f32<OT>(v);
        }
    }
}

// a 16-byte group of the row a thread for few rows, so that a row's loads are all in flight; fewer threads for many
int row_threads(int H, int n_rows) {
    const int most = n_rows > 256 ? 256 : 1024;
    int t = ((H + 3) / 4 + 31) & ~31;
    return t < 64 ? 64 : (t > most ? most : t);
}
size_t row_smem(int H) { return (size_t)(((H + 3) & ~3) + 33) * sizeof(float); }

template <typename K>
cudaError_t allow_smem(K k, size_t smem) {
    return smem > 48 * 1024 ? cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess;
}
}  // namespace

extern "C" int rb_add_layernorm(float* resid, const float* delta, int n_delta, long long delta_stride, const float* w,
                                const float* b, void* out, int out_dtype, const int* rows, int n_rows, int H, float eps,
                                int write_back, void* stream) {
    if (n_rows <= 0) return RB_OK;
    if (H <= 0 || !w || !out || n_delta < 0 || (n_delta > 0 && !delta)) return RB_ERR_BAD_SIZE;
    const size_t smem = row_smem(H);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    const size_t osz = out_dtype == RB_F32 ? 4 : 2;
    const int vec = (H & 3) == 0 && ((((uintptr_t)resid | (uintptr_t)delta | (uintptr_t)w | (uintptr_t)b) & 15) == 0) &&
                    ((uintptr_t)out & (4 * osz - 1)) == 0 && (n_delta <= 1 || (delta_stride & 3) == 0);
    cudaStream_t s = (cudaStream_t)stream;
#define RB_ALN(OT)                                                                                                        \
    do {                                                                                                                  \
        auto k = add_layernorm_kernel<OT>;                                                                                \
        cudaError_t e = allow_smem(k, smem);                                                                              \
        if (e != cudaSuccess) return (int)e;                                                                              \
        RB_LAUNCH((k), dim3(n_rows), dim3(row_threads(H, n_rows)), smem, s, resid, delta, n_delta, (size_t)delta_stride, w, b, \
                  (OT*)out, rows, H, eps, write_back, vec);                                                                \
    } while (0)
    if (out_dtype == RB_F32) RB_ALN(float);
    else if (out_dtype == RB_BF16) RB_ALN(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_ALN
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_out_norm(float* resid, const float* delta, int n_delta, long long delta_stride, float d_scale,
                           const int* row_of, const float* weights, int top, const float* self_weight, const void* self_x,
                           int self_dtype, int layer, const float* w, const float* b, float eps, float mult, void* out,
                           int out_dtype, int n_rows, int H, void* stream) {
    if (n_rows <= 0) return RB_OK;
    if (H <= 0 || !w || n_delta < 0 || ((n_delta > 0 || row_of) && !delta)) return RB_ERR_BAD_SIZE;
    if (row_of && (!weights || top < 1 || (self_weight && !self_x))) return RB_ERR_BAD_SIZE;
    const size_t smem = row_smem(H);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    const size_t osz = out_dtype == RB_F32 ? 4 : 2, xsz = self_dtype == RB_F32 ? 4 : 2;
    const int vec = (H & 3) == 0 && ((((uintptr_t)resid | (uintptr_t)delta | (uintptr_t)w | (uintptr_t)b) & 15) == 0) &&
                    ((uintptr_t)out & (4 * osz - 1)) == 0 && ((uintptr_t)self_x & (4 * xsz - 1)) == 0 && (delta_stride & 3) == 0;
    const Routed r{row_of, weights, top, row_of ? self_weight : nullptr};
    cudaStream_t s = (cudaStream_t)stream;
#define RB_ON(OT, XT)                                                                                                     \
    do {                                                                                                                  \
        auto k = out_norm_kernel<OT, XT>;                                                                                 \
        cudaError_t e = allow_smem(k, smem);                                                                              \
        if (e != cudaSuccess) return (int)e;                                                                              \
        RB_LAUNCH((k), dim3(n_rows), dim3(row_threads(H, n_rows)), smem, s, resid, delta, n_delta, (size_t)delta_stride,  \
                  d_scale, r, (const XT*)self_x, layer, w, b, eps, mult, (OT*)out, H, vec);                                \
    } while (0)
    const bool xf = !r.self_weight || self_dtype == RB_F32;
    if (!xf && self_dtype != RB_BF16) return RB_ERR_BAD_DTYPE;
    if (out && out_dtype == RB_BF16) { if (xf) RB_ON(__nv_bfloat16, float); else RB_ON(__nv_bfloat16, __nv_bfloat16); }
    else if (!out || out_dtype == RB_F32) { if (xf) RB_ON(float, float); else RB_ON(float, __nv_bfloat16); }
    else return RB_ERR_BAD_DTYPE;
#undef RB_ON
    RB_LAUNCH_CHECK();
    return RB_OK;
}

extern "C" int rb_pair_norm(const float* da, int na, long long sa, const float* db, int nb, long long sb, const float* wa, const float* wb,
                            float eps_in, float factor, float* out_v, float* resid, const float* w, float eps, float mult, void* out,
                            int out_dtype, int n_rows, int H, void* stream) {
    if (n_rows <= 0) return RB_OK;
    if (H <= 0 || !da || !db || na < 1 || nb < 1 || !wa || !wb || (w ? !resid : !out_v)) return RB_ERR_BAD_SIZE;
    const size_t smem = (size_t)(2 * ((H + 3) & ~3) + 66) * sizeof(float);
    if (smem > 200 * 1024) return RB_ERR_BAD_SIZE;
    const int vec = (H & 3) == 0 && (((uintptr_t)da | (uintptr_t)db) & 15) == 0 && ((sa | sb) & 3) == 0;
    int threads = (H + 31) & ~31;
    const int most = n_rows > 256 ? 256 : 1024;
    threads = threads < 64 ? 64 : (threads > most ? most : threads);
#define RB_PN(OT)                                                                                                                  \
    do {                                                                                                                           \
        auto k = pair_norm_kernel<OT>;                                                                                             \
        cudaError_t e = allow_smem(k, smem);                                                                                       \
        if (e != cudaSuccess) return (int)e;                                                                                       \
        RB_LAUNCH((k), dim3(n_rows), dim3(threads), smem, (cudaStream_t)stream, da, na, (size_t)sa, db, nb, (size_t)sb, wa, wb,    \
                  eps_in, factor, out_v, resid, w, eps, mult, (OT*)out, H, vec);                                                   \
    } while (0)
    if (!out || out_dtype == RB_F32) RB_PN(float);
    else if (out_dtype == RB_BF16) RB_PN(__nv_bfloat16);
    else return RB_ERR_BAD_DTYPE;
#undef RB_PN
    RB_LAUNCH_CHECK();
    return RB_OK;
}
