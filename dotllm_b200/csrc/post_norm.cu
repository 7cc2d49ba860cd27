// A norm behind the sum: the residual stream x and a sublayer's output y become
//
//   u = alpha x + y,   x <- u / sqrt(mean(u^2) + eps) * g          (g: one number for the whole row, or one per channel)
//
// in place, float32, with a copy in the type the next sublayer reads.  Two things may ride the same kernel:
//   * the model's last norm: the copy is x / sqrt(mean(x^2) + eps2) * g2 of the new x;
//   * in a step of one token per sequence, the next sublayer's input convolution: the copy is x + sum_j w_j x_(t-j) over the
//     row's own history (float32, K - 1 rows of the slot's memory, oldest first), which moves on by one row.
// Without y the stream is taken as it is (the first layer's input).
//
// One block per row; every thread keeps its values of the row in registers between the passes (rows of up to
// PN_THREADS * 4 * PN_MAX values that are a multiple of four), or walks them through memory (other widths).
#include "common.cuh"

#define PN_THREADS 256
#define PN_BIG 1024
#define PN_MAX 8

struct PnArgs {
    float* x;                    // [rows, width] contiguous
    const void* y;               // [rows, width], rows y_stride apart, or NULL
    int y_stride, y_bf16;
    float alpha, eps;
    const float* gain;           // [1] or [width]
    int gain_step;               // 0 or 1
    const float* gain2;          // the last norm's gain, or NULL
    int gain2_step;
    float eps2;
    void* out;                   // [rows, width] contiguous, or NULL
    int out_bf16, width;
    float* hist;                 // slot memory of the input convolution, or NULL: none
    long hist_stride;
    int n_slots;
    const int32_t* slots;        // [rows]
    const float* taps;           // [K, width], row K - 1 meets the current token
    int K;
};

__device__ __forceinline__ float4 pn_load_y(const PnArgs& a, size_t row, int c) {
    if (a.y_bf16) {
        const uint2 raw = *reinterpret_cast<const uint2*>((const __nv_bfloat16*)a.y + row * a.y_stride + c);
        const __nv_bfloat162 lo = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), hi = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
        return make_float4(__low2float(lo), __high2float(lo), __low2float(hi), __high2float(hi));
    }
    return *reinterpret_cast<const float4*>((const float*)a.y + row * a.y_stride + c);
}
__device__ __forceinline__ float pn_y(const PnArgs& a, size_t row, int c) {
    return a.y_bf16 ? __bfloat162float(((const __nv_bfloat16*)a.y)[row * a.y_stride + c]) : ((const float*)a.y)[row * a.y_stride + c];
}
__device__ __forceinline__ void pn_store4(const PnArgs& a, size_t at, float4 v) {
    if (a.out_bf16) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&lo);
        raw.y = *reinterpret_cast<uint32_t*>(&hi);
        *reinterpret_cast<uint2*>((__nv_bfloat16*)a.out + at) = raw;
    } else {
        *reinterpret_cast<float4*>((float*)a.out + at) = v;
    }
}
__device__ __forceinline__ void pn_store(const PnArgs& a, size_t at, float v) {
    if (a.out_bf16) ((__nv_bfloat16*)a.out)[at] = __float2bfloat16_rn(v);
    else ((float*)a.out)[at] = v;
}
__device__ __forceinline__ float4 pn_gain4(const float* gain, int step, int c) {
    if (step == 0) { const float g = gain[0]; return make_float4(g, g, g, g); }
    return *reinterpret_cast<const float4*>(gain + c);
}

// The row in registers: NV pieces of four per thread.  KT > 0: a convolution of up to KT taps whose taps and history are asked for
// together with the row, ahead of the norm's barriers; KT 0: none, or one of more taps, read where it is used.
template <int THREADS, int NV, int KT>
__global__ void __launch_bounds__(THREADS) post_norm_kernel(const PnArgs a) {
    __shared__ float scratch[33];
    dl_launch_dependents();
    const size_t row = blockIdx.x, base = row * a.width;
    const int tid = threadIdx.x;
    float4 tap[NV][KT > 0 ? KT : 1], past[NV][KT > 1 ? KT - 1 : 1];
    if (KT > 0) {                                            // weights: no kernel of the stream writes them
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < KT; ++j) {                   // place KT - 1 - lag meets the input `lag` rows back
                const int c = (tid + i * THREADS) * 4, at = a.K - KT + j;
                tap[i][j] = at >= 0 && c < a.width ? *reinterpret_cast<const float4*>(a.taps + (size_t)at * a.width + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    }
    dl_grid_dependency_wait();
    const int slot = a.hist != nullptr ? a.slots[row] : -1;
    const bool conv = slot >= 0 && slot < a.n_slots;
    float* hs = conv ? a.hist + (size_t)slot * a.hist_stride : nullptr;
    float4 u[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * THREADS) * 4;
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < a.width) {
            u[i] = *reinterpret_cast<const float4*>(a.x + base + c);
            if (KT > 1) {
#pragma unroll
                for (int j = 0; j + 1 < KT; ++j) {
                    const int at = a.K - KT + j;
                    past[i][j] = conv && at >= 0 ? *reinterpret_cast<const float4*>(hs + (size_t)at * a.width + c) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
            if (a.y != nullptr) {
                const float4 y = pn_load_y(a, row, c);
                u[i] = make_float4(fmaf(a.alpha, u[i].x, y.x), fmaf(a.alpha, u[i].y, y.y), fmaf(a.alpha, u[i].z, y.z), fmaf(a.alpha, u[i].w, y.w));
            }
        }
        ss += (u[i].x * u[i].x + u[i].y * u[i].y) + (u[i].z * u[i].z + u[i].w * u[i].w);
    }
    if (a.y != nullptr) {
        ss = dl_block_sum(ss, scratch);
        const float r = 1.0f / sqrtf(ss / (float)a.width + a.eps);
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (tid + i * THREADS) * 4;
            if (c < a.width) {
                const float4 g = pn_gain4(a.gain, a.gain_step, c);
                u[i] = make_float4(u[i].x * r * g.x, u[i].y * r * g.y, u[i].z * r * g.z, u[i].w * r * g.w);
                *reinterpret_cast<float4*>(a.x + base + c) = u[i];
            }
            ss += (u[i].x * u[i].x + u[i].y * u[i].y) + (u[i].z * u[i].z + u[i].w * u[i].w);
        }
    }
    if (a.gain2 != nullptr) {
        ss = dl_block_sum(ss, scratch);
        const float r = 1.0f / sqrtf(ss / (float)a.width + a.eps2);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (tid + i * THREADS) * 4;
            if (c < a.width) {
                const float4 g = pn_gain4(a.gain2, a.gain2_step, c);
                pn_store4(a, base + c, make_float4(u[i].x * r * g.x, u[i].y * r * g.y, u[i].z * r * g.z, u[i].w * r * g.w));
            }
        }
        return;
    }
    if (a.out == nullptr) return;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * THREADS) * 4;
        if (c >= a.width) continue;
        float4 h = u[i];
        if (conv) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            if (KT > 0) {
#pragma unroll
                for (int j = 0; j < KT; ++j) {                   // oldest first; a history row moves to the place before it
                    const float4 w = tap[i][j], in = j + 1 < KT ? past[i][j] : u[i];
                    const int at = a.K - KT + j;
                    if (at > 0) *reinterpret_cast<float4*>(hs + (size_t)(at - 1) * a.width + c) = in;
                    acc = make_float4(fmaf(w.x, in.x, acc.x), fmaf(w.y, in.y, acc.y), fmaf(w.z, in.z, acc.z), fmaf(w.w, in.w, acc.w));
                }
            } else {
                for (int j = 0; j < a.K; ++j) {
                    const float4 w = *reinterpret_cast<const float4*>(a.taps + (size_t)j * a.width + c);
                    const float4 in = j + 1 < a.K ? *reinterpret_cast<const float4*>(hs + (size_t)j * a.width + c) : u[i];
                    if (j > 0) *reinterpret_cast<float4*>(hs + (size_t)(j - 1) * a.width + c) = in;
                    acc = make_float4(fmaf(w.x, in.x, acc.x), fmaf(w.y, in.y, acc.y), fmaf(w.z, in.z, acc.z), fmaf(w.w, in.w, acc.w));
                }
            }
            h = make_float4(h.x + acc.x, h.y + acc.y, h.z + acc.z, h.w + acc.w);
        }
        pn_store4(a, base + c, h);
    }
}

// Any width: the row goes through memory (every value is read and written by one thread alone).
__global__ void __launch_bounds__(PN_THREADS) post_norm_wide_kernel(const PnArgs a) {
    __shared__ float scratch[33];
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const size_t row = blockIdx.x, base = row * a.width;
    float ss = 0.f;
    for (int c = threadIdx.x; c < a.width; c += PN_THREADS) {
        float v = a.x[base + c];
        if (a.y != nullptr) v = fmaf(a.alpha, v, pn_y(a, row, c));
        ss += v * v;
    }
    if (a.y != nullptr) {
        ss = dl_block_sum(ss, scratch);
        const float r = 1.0f / sqrtf(ss / (float)a.width + a.eps);
        ss = 0.f;
        for (int c = threadIdx.x; c < a.width; c += PN_THREADS) {
            const float v = fmaf(a.alpha, a.x[base + c], pn_y(a, row, c)) * r * a.gain[a.gain_step ? c : 0];
            a.x[base + c] = v;
            ss += v * v;
        }
    }
    if (a.gain2 != nullptr) {
        ss = dl_block_sum(ss, scratch);
        const float r = 1.0f / sqrtf(ss / (float)a.width + a.eps2);
        for (int c = threadIdx.x; c < a.width; c += PN_THREADS) pn_store(a, base + c, a.x[base + c] * r * a.gain2[a.gain2_step ? c : 0]);
        return;
    }
    if (a.out == nullptr) return;
    const int slot = a.hist != nullptr ? a.slots[row] : -1;
    const bool conv = slot >= 0 && slot < a.n_slots;
    float* hs = conv ? a.hist + (size_t)slot * a.hist_stride : nullptr;
    for (int c = threadIdx.x; c < a.width; c += PN_THREADS) {
        const float v = a.x[base + c];
        float h = v;
        if (conv) {
            float acc = 0.f;
            for (int j = 0; j < a.K; ++j) {
                const float in = j + 1 < a.K ? hs[(size_t)j * a.width + c] : v;
                if (j > 0) hs[(size_t)(j - 1) * a.width + c] = in;
                acc = fmaf(a.taps[(size_t)j * a.width + c], in, acc);
            }
            h += acc;
        }
        pn_store(a, base + c, h);
    }
}

// x float32 [rows, width] contiguous, updated in place; y [rows, width] of y_dtype (rows y_stride apart) or NULL; gain float32
// of gain_n = 1 or width values; gain2 likewise or NULL; out contiguous of out_dtype or NULL.  hist (float32 slot memory,
// hist_stride floats a slot, its first (K - 1) * width the convolution's last inputs) or NULL; slots int32 [rows];
// taps float32 [K, width].  With hist every row must be the only row of its sequence in the step.
extern "C" int dl_post_norm(float* x, const void* y, int y_dtype, int y_stride, float alpha, const float* gain, int gain_n,
                            float eps, const float* gain2, int gain2_n, float eps2, void* out, int out_dtype, int rows, int width,
                            float* hist, long hist_stride, int n_slots, const int32_t* slots, const float* taps, int K,
                            void* stream) {
    DL_REQUIRE(rows >= 0 && width > 0, "post_norm: bad sizes rows=%d width=%d", rows, width);
    DL_REQUIRE(y == nullptr || ((y_dtype == DL_F32 || y_dtype == DL_BF16) && y_stride >= width && gain != nullptr && eps > 0.f),
               "post_norm: what joins the stream needs a type, whole rows, a gain and a positive eps");
    DL_REQUIRE((y == nullptr || gain_n == 1 || gain_n == width) && (gain2 == nullptr || gain2_n == 1 || gain2_n == width),
               "post_norm: a gain holds one value or one per channel");
    DL_REQUIRE(gain2 == nullptr || (out != nullptr && eps2 > 0.f && hist == nullptr), "post_norm: the last norm writes a copy, without a convolution");
    DL_REQUIRE(out == nullptr || out_dtype == DL_F32 || out_dtype == DL_BF16, "post_norm: out dtype %d", out_dtype);
    DL_REQUIRE(hist == nullptr || (K >= 1 && taps != nullptr && slots != nullptr && n_slots > 0 && out != nullptr && hist_stride >= (long)(K - 1) * width),
               "post_norm: an input convolution needs taps, slots, memory and a copy to write");
    if (rows == 0) return DL_OK;
    PnArgs a = {x, y, y_stride, y_dtype == DL_BF16 ? 1 : 0, alpha, eps, gain, gain_n == 1 ? 0 : 1, gain2, gain2_n == 1 ? 0 : 1, eps2,
                out, out_dtype == DL_BF16 ? 1 : 0, width, hist, hist_stride, n_slots, slots, taps, K};
    const auto al16 = [](const void* p) { return ((uintptr_t)p % 16) == 0; };
    const bool vec = width % 4 == 0 && width <= PN_THREADS * 4 * PN_MAX && al16(x) && (y == nullptr || (al16(y) && y_stride % 4 == 0)) &&
                     (out == nullptr || al16(out)) && (hist == nullptr || (al16(hist) && hist_stride % 4 == 0 && al16(taps))) &&
                     (y == nullptr || gain_n == 1 || al16(gain)) && (gain2 == nullptr || gain2_n == 1 || al16(gain2));
    // few rows (a decode step): as many threads as a row has pieces, up to 1,024
    const bool big = rows <= 2 * dl_sm_count() && width > PN_THREADS * 4;
    const int threads = big ? PN_BIG : PN_THREADS, pieces = (width / 4 + threads - 1) / threads;
    const bool short_conv = hist != nullptr && K <= 4;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
    const dim3 grid(rows), block(vec ? threads : PN_THREADS);
#define PN_GO(T, NV, KT) e = dl_launch_dependent(post_norm_kernel<T, NV, KT>, grid, block, 0, s, a)
    if (!vec) e = dl_launch_dependent(post_norm_wide_kernel, grid, block, 0, s, a);
    else if (big && pieces <= 1 && short_conv) PN_GO(PN_BIG, 1, 4);
    else if (big && pieces <= 1) PN_GO(PN_BIG, 1, 0);
    else if (big) PN_GO(PN_BIG, 2, 0);
    else if (pieces <= 1 && short_conv) PN_GO(PN_THREADS, 1, 4);
    else if (pieces <= 1) PN_GO(PN_THREADS, 1, 0);
    else if (pieces <= 2) PN_GO(PN_THREADS, 2, 0);
    else if (pieces <= 4) PN_GO(PN_THREADS, 4, 0);
    else PN_GO(PN_THREADS, PN_MAX, 0);
#undef PN_GO
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "post_norm: %s", cudaGetErrorString(e));
    return DL_OK;
}
