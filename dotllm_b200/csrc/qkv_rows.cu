// What stands between the stacked query/key/value product of an attention and its cache, in one kernel over the rows:
//
//   q' = norm_all(q + bq) * gq      k' = norm_all(k + bk) * gk      v' = (1 - w) (v + bv) + w v_first
//
// norm_all divides a row's part by its root mean square over ALL its heads (eps inside the root).  Biases, norms (gains NULL: no
// norm) and the mixing (v_first NULL: none) are each optional; w is one number on the device.  The row of x is [q | k | v] with
// heads d, d and vd wide; in the output every head of q and k is lay_k and every head of v lay_v wide, zeros behind its own
// values (a width that the tensor-core attention kernels take).  v_first holds heads first_lay apart: another layer's values of
// the same tokens, as this kernel wrote them there.
//
// Grid: (row, part).  A part's values are read once, 16 bytes a thread at a time where everything is aligned for it (VEC), and kept
// in registers across the reduction.  All arithmetic is float32, in an order fixed by the part's width.
#include "common.cuh"

#define QR_THREADS 256
#define QR_KEEP 32                       // values of a part a thread keeps in registers

struct QrPart {
    const float* bias;
    const float* gain;
    int heads, width, lay, from, to;     // heads of `width` values, `lay` apart in the output; first column in x and in the output
};

template <typename T, bool VEC>
__global__ void __launch_bounds__(QR_THREADS)
qkv_rows_kernel(const T* __restrict__ x, int ld, const QrPart qp, const QrPart kp, const QrPart vp, float eps, const T* __restrict__ first,
                int first_ld, int first_lay, const float* __restrict__ mix, T* __restrict__ out, int out_ld) {
    constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
    constexpr int NP = QR_KEEP / V;
    __shared__ float scratch[33];
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const size_t t = blockIdx.x;
    const QrPart p = blockIdx.y == 0 ? qp : (blockIdx.y == 1 ? kp : vp);
    const int n = p.heads * p.width;
    const T* src = x + t * ld + p.from;
    T* dst = out + t * out_ld + p.to;
    const bool mixes = blockIdx.y == 2 && first != nullptr;
    const float w = mixes ? *mix : 0.f;
    const T* other = mixes ? first + t * first_ld : nullptr;
    auto place = [&](int c) { return p.lay == p.width ? c : (c / p.width) * p.lay + c % p.width; };

    auto load = [&](int c, float (&f)[V]) {
        if (VEC) {
            const uint4 raw = *reinterpret_cast<const uint4*>(src + c);
            const T* r = reinterpret_cast<const T*>(&raw);
#pragma unroll
            for (int e = 0; e < V; ++e) f[e] = dl_to_f32<T>(r[e]);
            if (p.bias != nullptr) {
#pragma unroll
                for (int e = 0; e < V; e += 4) {
                    const float4 b = *reinterpret_cast<const float4*>(p.bias + c + e);
                    f[e % V] += b.x, f[(e + 1) % V] += b.y, f[(e + 2) % V] += b.z, f[(e + 3) % V] += b.w;
                }
            }
        } else {
            f[0] = dl_to_f32<T>(src[c]) + (p.bias != nullptr ? p.bias[c] : 0.f);
        }
    };
    auto store = [&](int c, float (&f)[V], float factor) {
        if (p.gain != nullptr) {
            if (VEC) {
#pragma unroll
                for (int e = 0; e < V; e += 4) {
                    const float4 g = *reinterpret_cast<const float4*>(p.gain + c + e);
                    f[e % V] *= factor * g.x, f[(e + 1) % V] *= factor * g.y, f[(e + 2) % V] *= factor * g.z, f[(e + 3) % V] *= factor * g.w;
                }
            } else {
                f[0] *= factor * p.gain[c];
            }
        }
        if (mixes) {
            const T* o = other + (c / p.width) * first_lay + c % p.width;
            if (VEC) {
                const uint4 raw = *reinterpret_cast<const uint4*>(o);
                const T* r = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int e = 0; e < V; ++e) f[e] = (1.f - w) * f[e] + w * dl_to_f32<T>(r[e]);
            } else {
                f[0] = (1.f - w) * f[0] + w * dl_to_f32<T>(*o);
            }
        }
        if (VEC) {
            uint4 raw;
            T* r = reinterpret_cast<T*>(&raw);
#pragma unroll
            for (int e = 0; e < V; ++e) r[e] = dl_from_f32<T>(f[e]);
            *reinterpret_cast<uint4*>(dst + place(c)) = raw;
        } else {
            dst[place(c)] = dl_from_f32<T>(f[0]);
        }
    };

    if (p.lay > p.width) {                                   // zeros behind every head
        const int pad = p.lay - p.width;
        for (int i = threadIdx.x; i < p.heads * pad; i += QR_THREADS) dst[(i / pad) * p.lay + p.width + i % pad] = dl_from_f32<T>(0.f);
    }
    const int step = QR_THREADS * V;
    if (p.gain == nullptr) {
        for (int c = threadIdx.x * V; c < n; c += step) {
            float f[V];
            load(c, f);
            store(c, f, 1.f);
        }
        return;
    }
    const bool keep = n <= QR_THREADS * QR_KEEP;
    float f[NP][V];
    float ss = 0.f;
    if (keep) {
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int c = (threadIdx.x + i * QR_THREADS) * V;
#pragma unroll
            for (int e = 0; e < V; ++e) f[i][e] = 0.f;
            if (c < n) load(c, f[i]);
#pragma unroll
            for (int e = 0; e < V; ++e) ss += f[i][e] * f[i][e];
        }
    } else {
        for (int c = threadIdx.x * V; c < n; c += step) {
            float g[V];
            load(c, g);
#pragma unroll
            for (int e = 0; e < V; ++e) ss += g[e] * g[e];
        }
    }
    ss = dl_block_sum(ss, scratch);
    const float factor = 1.0f / sqrtf(ss / (float)n + eps);
    if (keep) {
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int c = (threadIdx.x + i * QR_THREADS) * V;
            if (c < n) store(c, f[i], factor);
        }
    } else {
        for (int c = threadIdx.x * V; c < n; c += step) {
            float g[V];
            load(c, g);
            store(c, g, factor);
        }
    }
}

// x [rows, H*d + G*d + G*vd] of dtype, rows ld apart; biases float32 (q_bias [H*d], k_bias [G*d], v_bias [G*vd], each or NULL);
// q_gain, k_gain float32 of the same widths, both or neither; first [rows, G*first_lay] of dtype (rows first_ld apart) with mix
// float32 [1], or both NULL; out [rows, H*lay_k + G*lay_k + G*lay_v] of dtype, rows out_ld apart.
extern "C" int dl_qkv_rows(const void* x, int dtype, int ld, const float* q_bias, const float* k_bias, const float* v_bias,
                           const float* q_gain, const float* k_gain, float eps, int H, int G, int d, int vd, int lay_k, int lay_v,
                           const void* first, int first_ld, int first_lay, const float* mix, void* out, int out_ld, int rows,
                           void* stream) {
    DL_REQUIRE(rows >= 0 && H > 0 && G > 0 && d > 0 && vd > 0 && lay_k >= d && lay_v >= vd, "qkv_rows: bad sizes");
    DL_REQUIRE(ld >= H * d + G * (d + vd) && out_ld >= H * lay_k + G * (lay_k + lay_v), "qkv_rows: rows too short");
    DL_REQUIRE(dtype == DL_F32 || dtype == DL_BF16, "qkv_rows: dtype %d", dtype);
    DL_REQUIRE((q_gain == nullptr) == (k_gain == nullptr) && (q_gain == nullptr || eps > 0.f), "qkv_rows: both norms or neither, eps positive");
    DL_REQUIRE((first == nullptr) == (mix == nullptr) && (first == nullptr || (first_lay >= vd && first_ld >= (G - 1) * first_lay + vd)),
               "qkv_rows: mixed values need the other values, wide enough, and their weight");
    if (rows == 0) return DL_OK;
    const int v = dtype == DL_BF16 ? 8 : 4;
    const uintptr_t places = (uintptr_t)x | (uintptr_t)q_bias | (uintptr_t)k_bias | (uintptr_t)v_bias | (uintptr_t)q_gain | (uintptr_t)k_gain |
                             (uintptr_t)first | (uintptr_t)out;
    const bool vec = places % 16 == 0 && ld % v == 0 && out_ld % v == 0 && d % v == 0 && vd % v == 0 && lay_k % v == 0 && lay_v % v == 0 &&
                     (first == nullptr || (first_ld % v == 0 && first_lay % v == 0));
    const QrPart qp{q_bias, q_gain, H, d, lay_k, 0, 0};
    const QrPart kp{k_bias, k_gain, G, d, lay_k, H * d, H * lay_k};
    const QrPart vp{v_bias, nullptr, G, vd, lay_v, (H + G) * d, (H + G) * lay_k};
    const dim3 grid(rows, 3), block(QR_THREADS);
    cudaError_t e;
#define QR_GO(T, VEC)                                                                                                                     \
    e = dl_launch_dependent(qkv_rows_kernel<T, VEC>, grid, block, 0, (cudaStream_t)stream, (const T*)x, ld, qp, kp, vp, eps, (const T*)first, \
                            first_ld, first_lay, mix, (T*)out, out_ld)
    if (dtype == DL_F32) { if (vec) QR_GO(float, true); else QR_GO(float, false); }
    else { if (vec) QR_GO(__nv_bfloat16, true); else QR_GO(__nv_bfloat16, false); }
#undef QR_GO
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "qkv_rows: %s", cudaGetErrorString(e));
    return DL_OK;
}
