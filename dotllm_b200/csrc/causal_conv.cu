// A short causal convolution over time per channel, with the last inputs of every sequence kept from step to step:
//
//   y_t[c] = act(bias[c] + sum_j taps[j][c] x_(t - K + 1 + j)[c])  (+ x_t[c])        zeros before the sequence's start
//
// x: rows of a step's packed tokens (float32 or bfloat16); sums, bias, activation and history are float32.  A sequence's last
// K - 1 inputs lie in its slot's memory, oldest first.  The grid is (runs of tokens of a sequence, channels, sequences): a
// thread owns VEC neighbouring channels, keeps their taps and last inputs in registers and walks its run.  A run is at least K - 1
// tokens long, so the old history is read by a sequence's first run alone; that run's threads also leave the new history
// (they read the sequence's last inputs again), which is why one kernel does both without a race.
#include "common.cuh"

#define CC_THREADS 128
#define CC_MAX_TAPS 64

template <typename T, int VEC>
__device__ __forceinline__ void cc_load(const T* p, float (&o)[VEC]) {
    if (VEC == 1) { o[0] = dl_to_f32<T>(p[0]); return; }
    if (sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
        const float f[4] = {__low2float(a), __high2float(a), __low2float(b), __high2float(b)};
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = f[e & 3];
    } else {
        const float4 raw = *reinterpret_cast<const float4*>(p);
        const float f[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
        for (int e = 0; e < VEC; ++e) o[e] = f[e & 3];
    }
}
template <typename T, int VEC>
__device__ __forceinline__ void cc_store(T* p, const float (&o)[VEC]) {
    if (VEC == 1) { p[0] = dl_from_f32<T>(o[0]); return; }
    if (sizeof(T) == 2) {
        __nv_bfloat162 a = __floats2bfloat162_rn(o[0], o[1 % VEC]), b = __floats2bfloat162_rn(o[2 % VEC], o[3 % VEC]);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    } else {
        *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1 % VEC], o[2 % VEC], o[3 % VEC]);
    }
}

template <typename T, typename TO, int KMAX, int VEC>
__global__ void __launch_bounds__(CC_THREADS)
causal_conv_kernel(const T* __restrict__ x, int ld, const float* __restrict__ taps, int K, const float* __restrict__ bias, int silu,
                   int add_input, float* __restrict__ hist, long hist_stride, int n_slots, const int32_t* __restrict__ cu_new,
                   const int32_t* __restrict__ slots, TO* __restrict__ out, int out_ld, int C, int run) {
    dl_launch_dependents();
    const int c = (blockIdx.y * CC_THREADS + threadIdx.x) * VEC;
    float tap[KMAX][VEC], in[KMAX][VEC], b4[VEC];
    if (c < C) {                                             // weights: no kernel of the stream writes them
#pragma unroll
        for (int i = 0; i < KMAX; ++i) {                     // place KMAX - 1 - lag meets the input `lag` tokens back
            const int lag = KMAX - 1 - i;
#pragma unroll
            for (int e = 0; e < VEC; ++e) tap[i][e] = 0.f, in[i][e] = 0.f;
            if (lag < K) cc_load<float, VEC>(taps + (size_t)(K - 1 - lag) * C + c, tap[i]);
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) b4[e] = 0.f;
        if (bias != nullptr) cc_load<float, VEC>(bias + c, b4);
    }
    dl_grid_dependency_wait();
    const int seq = blockIdx.z;
    const int t0 = cu_new[seq], n = cu_new[seq + 1] - t0;
    const int j0 = blockIdx.x * run, j1 = min(n, j0 + run);
    const int slot = slots[seq];
    if (c >= C || j0 >= n || slot < 0 || slot >= n_slots) return;
    float* hs = hist + (size_t)slot * hist_stride;
    const T* xs = x + (size_t)t0 * ld + c;
#pragma unroll
    for (int lag = 1; lag < KMAX; ++lag) {
        if (lag >= K) continue;
        const int j = j0 - lag;                              // among the step's inputs, or in the history, whose row K - 2 is the newest
        if (j >= 0) cc_load<T, VEC>(xs + (size_t)j * ld, in[KMAX - 1 - lag]);
        else cc_load<float, VEC>(hs + (size_t)(K - 1 + j) * C + c, in[KMAX - 1 - lag]);
    }
    float ahead[VEC];
    cc_load<T, VEC>(xs + (size_t)j0 * ld, ahead);
    for (int j = j0; j < j1; ++j) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) in[KMAX - 1][e] = ahead[e];
        if (j + 1 < j1) cc_load<T, VEC>(xs + (size_t)(j + 1) * ld, ahead);
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            float acc = 0.f;
#pragma unroll
            for (int i = 0; i < KMAX; ++i) acc = fmaf(tap[i][e], in[i][e], acc);     // oldest first; a place in front of the taps adds 0 * 0
            acc += b4[e];
            if (silu) acc = acc / (1.0f + expf(-acc));
            y[e] = add_input ? in[KMAX - 1][e] + acc : acc;
        }
        cc_store<TO, VEC>(out + (size_t)(t0 + j) * out_ld + c, y);
#pragma unroll
        for (int i = 0; i + 1 < KMAX; ++i)
#pragma unroll
            for (int e = 0; e < VEC; ++e) in[i][e] = in[i + 1][e];
    }
    if (j0 == 0) {                                           // the sequence's first run: the only reader of the old history
        for (int i = 0; i < K - 1; ++i) {                    // ascending: a place is read (at i + n) before it is written
            const int src = i + n;                           // index in (old history ++ new inputs)
            float v[VEC];
            if (src < K - 1) cc_load<float, VEC>(hs + (size_t)src * C + c, v);
            else cc_load<T, VEC>(xs + (size_t)(src - (K - 1)) * ld, v);
            cc_store<float, VEC>(hs + (size_t)i * C + c, v);
        }
    }
}

template <typename T, typename TO>
static cudaError_t cc_launch(const void* x, int ld, const float* taps, int K, const float* bias, int silu, int add_input, float* hist,
                             long hist_stride, int n_slots, const int32_t* cu_new, const int32_t* slots, void* out, int out_ld,
                             int n_seqs, int max_new, int C, cudaStream_t s) {
    const bool vec = C % 4 == 0 && ld % 4 == 0 && out_ld % 4 == 0 && hist_stride % 4 == 0 && ((uintptr_t)x % (4 * sizeof(T))) == 0 &&
                     ((uintptr_t)out % (4 * sizeof(TO))) == 0 && ((uintptr_t)hist % 16) == 0 && ((uintptr_t)taps % 16) == 0 &&
                     (bias == nullptr || ((uintptr_t)bias % 16) == 0) && K <= 16;
    const int per = CC_THREADS * (vec ? 4 : 1), chunks = (C + per - 1) / per;
    // runs: long ones read few inputs twice, short ones fill the machine
    int run = 8;
    while (run < 32 && (long)n_seqs * chunks * ((max_new + 2 * run - 1) / (2 * run)) >= 148 * 16) run *= 2;
    if (run < K - 1) run = K - 1;
    const dim3 grid((max_new + run - 1) / run, chunks, n_seqs), block(CC_THREADS);
#define CC_GO(KMAX, VEC)                                                                                                    \
    return dl_launch_dependent(causal_conv_kernel<T, TO, KMAX, VEC>, grid, block, 0, s, (const T*)x, ld, taps, K, bias, silu, \
                               add_input, hist, hist_stride, n_slots, cu_new, slots, (TO*)out, out_ld, C, run)
    if (vec) {
        if (K <= 4) CC_GO(4, 4);
        if (K <= 8) CC_GO(8, 4);
        CC_GO(16, 4);
    }
    if (K <= 4) CC_GO(4, 1);
    if (K <= 16) CC_GO(16, 1);
    CC_GO(CC_MAX_TAPS, 1);
#undef CC_GO
}

// x [tokens, C] of dtype (rows ld apart), taps float32 [K, C] (row K - 1 meets the current token), bias float32 [C] or NULL;
// silu: 1 for silu behind the sum; add_input: 1 adds x_t; hist float32, hist_stride floats a slot, the first (K - 1) * C the
// last inputs; cu_new int32 [n_seqs + 1]; slots int32 [n_seqs]; max_new: the most tokens a sequence brings; out [tokens, C] of
// out_dtype (rows out_ld apart).
extern "C" int dl_causal_conv(const void* x, int dtype, int ld, const float* taps, int K, const float* bias, int silu, int add_input,
                              float* hist, long hist_stride, int n_slots, const int32_t* cu_new, const int32_t* slots, void* out,
                              int out_dtype, int out_ld, int n_seqs, int max_new, int C, void* stream) {
    DL_REQUIRE(n_seqs >= 0 && max_new >= 0 && C > 0 && K >= 1 && n_slots > 0, "causal_conv: bad sizes");
    DL_REQUIRE(K <= CC_MAX_TAPS, "causal_conv: %d taps, the kernel takes up to %d", K, CC_MAX_TAPS);
    DL_REQUIRE(ld >= C && out_ld >= C && (K == 1 || hist_stride >= (long)(K - 1) * C) && n_seqs <= 65535, "causal_conv: rows overlap or too many sequences");
    DL_REQUIRE((dtype == DL_F32 || dtype == DL_BF16) && (out_dtype == DL_F32 || out_dtype == DL_BF16), "causal_conv: dtypes %d, %d", dtype, out_dtype);
    if (n_seqs == 0 || max_new == 0) return DL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    cudaError_t e;
#define CC_TYPES(T, TO) e = cc_launch<T, TO>(x, ld, taps, K, bias, silu, add_input, hist, hist_stride, n_slots, cu_new, slots, out, out_ld, n_seqs, max_new, C, s)
    if (dtype == DL_F32 && out_dtype == DL_F32) CC_TYPES(float, float);
    else if (dtype == DL_F32) CC_TYPES(float, __nv_bfloat16);
    else if (out_dtype == DL_F32) CC_TYPES(__nv_bfloat16, float);
    else CC_TYPES(__nv_bfloat16, __nv_bfloat16);
#undef CC_TYPES
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "causal_conv: %s", cudaGetErrorString(e));
    return DL_OK;
}
