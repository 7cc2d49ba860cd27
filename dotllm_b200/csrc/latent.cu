// The small steps around attention over a latent that all heads share (parts/latent_attention.py), and the gate per channel.
//
// dl_latent_rows: from the stacked projection's row [query latent | key/value latent | rotated key part] the two latents, each
// divided by its root mean square and multiplied by its gain, and the key part rotated by the token's position; the second latent
// and the key part go side by side into one row of `lay` values (zeros behind them): what the cache keeps of the token.
// dl_latent_query_tail: the queries' rotated parts.  Head h of q holds [dim | rot] channels; channels dim .. dim + rot are
// rotated into channels rank .. rank + rot of head h of out (lay wide), and zeros go behind them.
// dl_channel_gate: out[t, h, c] = scale * o[t, h, c] * sigmoid(g[t, h, c]) for heads laid out `lay` >= width apart in o (g NULL: no
// gate, the scale alone).
// Rotations pair channel 2i with 2i + 1 (the first rot_dims of a part; the rest pass unchanged).  All arithmetic is float32.
#include "common.cuh"

__device__ __forceinline__ void lt_pair(float u, float v, float c, float s, float& a, float& b) {
    a = u * c - v * s;
    b = v * c + u * s;
}

// Channel c of a part of `rot` channels, its first rot_dims rotated; zeros beyond.
template <typename T>
__device__ __forceinline__ float lt_tail(const T* __restrict__ src, int c, int rot, int rot_dims, const float* __restrict__ cos_t,
                                         const float* __restrict__ sin_t, int pos) {
    if (c >= rot) return 0.f;
    const float v = dl_to_f32<T>(src[c]);
    if (c >= rot_dims) return v;
    const size_t at = (size_t)pos * (rot_dims / 2) + (c >> 1);
    const float other = dl_to_f32<T>(src[c ^ 1]), cs = cos_t[at], sn = sin_t[at];
    float a, b;
    lt_pair(c & 1 ? other : v, c & 1 ? v : other, cs, sn, a, b);
    return c & 1 ? b : a;
}

#define LT_THREADS 128
#define LT_KEEP 16                       // values of a latent a thread keeps in registers

// Eight (bfloat16) or four (float32) neighbours at a time where everything is aligned for it (VEC), else one.
template <typename T, bool VEC>
__global__ void __launch_bounds__(LT_THREADS)
latent_rows_kernel(const T* __restrict__ x, int ld, int q_rank, int kv_rank, int rot, int rot_dims, const float* __restrict__ q_gain,
                   const float* __restrict__ kv_gain, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                   int table_rows, const int32_t* __restrict__ token_pos, T* __restrict__ q_out, T* __restrict__ kv_out, int lay) {
    constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
    __shared__ float scratch[33];
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const size_t t = blockIdx.x;
    const bool is_q = blockIdx.y == 1;
    const int rank = is_q ? q_rank : kv_rank;
    const T* src = x + t * ld + (is_q ? 0 : q_rank);
    T* dst = is_q ? q_out + t * q_rank : kv_out + t * lay;
    const float* gain = is_q ? q_gain : kv_gain;
    if (!is_q) {                                             // the part behind the latent: it waits for no sum
        const int pos = rot_dims > 0 ? min(token_pos[t], table_rows - 1) : 0;    // host-validated
        for (int c = threadIdx.x; c < lay - kv_rank; c += LT_THREADS)
            dst[kv_rank + c] = dl_from_f32<T>(lt_tail<T>(src + kv_rank, c, rot, rot_dims, cos_t, sin_t, pos));
    }
    const bool keep = rank <= LT_THREADS * LT_KEEP;
    float v[LT_KEEP];
    float ss = 0.f;
    if (keep) {
#pragma unroll
        for (int i = 0; i < LT_KEEP / V; ++i) {
            const int c = (threadIdx.x + i * LT_THREADS) * V;
            if (VEC) {
                uint4 raw = make_uint4(0u, 0u, 0u, 0u);
                if (c < rank) raw = *reinterpret_cast<const uint4*>(src + c);
                const T* r8 = reinterpret_cast<const T*>(&raw);
#pragma unroll
                for (int e = 0; e < V; ++e) v[i * V + e] = dl_to_f32<T>(r8[e]);
            } else {
                v[i] = c < rank ? dl_to_f32<T>(src[c]) : 0.f;
            }
#pragma unroll
            for (int e = 0; e < V; ++e) ss += v[i * V + e] * v[i * V + e];
        }
    } else {
        for (int c = threadIdx.x; c < rank; c += LT_THREADS) { const float w = dl_to_f32<T>(src[c]); ss += w * w; }
    }
    ss = dl_block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)rank + eps);
    if (keep) {
#pragma unroll
        for (int i = 0; i < LT_KEEP / V; ++i) {
            const int c = (threadIdx.x + i * LT_THREADS) * V;
            if (c >= rank) continue;
            if (VEC) {
                uint4 raw;
                T* r8 = reinterpret_cast<T*>(&raw);
#pragma unroll
                for (int e = 0; e < V; ++e) r8[e] = dl_from_f32<T>(v[i * V + e] * r * gain[c + e]);
                *reinterpret_cast<uint4*>(dst + c) = raw;
            } else {
                dst[c] = dl_from_f32<T>(v[i] * r * gain[c]);
            }
        }
    } else {
        for (int c = threadIdx.x; c < rank; c += LT_THREADS) dst[c] = dl_from_f32<T>(dl_to_f32<T>(src[c]) * r * gain[c]);
    }
}

// The same with a warp per (token, latent) and no block barrier: latents of up to 32 lanes x NP pieces of 16 bytes, aligned.
template <typename T, int NP>
__global__ void __launch_bounds__(LT_THREADS)
latent_rows_warp_kernel(const T* __restrict__ x, int ld, int q_rank, int kv_rank, int rot, int rot_dims, const float* __restrict__ q_gain,
                        const float* __restrict__ kv_gain, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                        int table_rows, const int32_t* __restrict__ token_pos, T* __restrict__ q_out, T* __restrict__ kv_out, int lay, int n_tokens) {
    constexpr int V = 16 / (int)sizeof(T);
    dl_launch_dependents();
    const int lane = threadIdx.x & 31, which = blockIdx.y;   // 0: the key/value latent and what lies behind it, 1: the query latent
    const int t = blockIdx.x * (LT_THREADS / 32) + (threadIdx.x >> 5);
    if (t >= n_tokens) return;
    const int rank = which ? q_rank : kv_rank;
    const float* gain = which ? q_gain : kv_gain;
    float gg[NP <= 4 ? NP * V : 1];
    if (NP <= 4) {                                           // weights: no kernel of the stream writes them
#pragma unroll
        for (int i = 0; i < NP; ++i)
#pragma unroll
            for (int e = 0; e < V; e += 4) {
                const int c = (lane + 32 * i) * V + e;
                const float4 w = c < rank ? *reinterpret_cast<const float4*>(gain + c) : make_float4(0.f, 0.f, 0.f, 0.f);
                gg[(i * V + e) % (NP * V)] = w.x, gg[(i * V + e + 1) % (NP * V)] = w.y, gg[(i * V + e + 2) % (NP * V)] = w.z, gg[(i * V + e + 3) % (NP * V)] = w.w;
            }
    }
    dl_grid_dependency_wait();
    const T* src = x + (size_t)t * ld + (which ? 0 : q_rank);
    T* dst = which ? q_out + (size_t)t * q_rank : kv_out + (size_t)t * lay;
    uint4 raw[NP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int c = (lane + 32 * i) * V;
        raw[i] = c < rank ? *reinterpret_cast<const uint4*>(src + c) : make_uint4(0u, 0u, 0u, 0u);
    }
    if (which == 0) {                                        // the part behind the latent: it waits for no sum
        const int pos = rot_dims > 0 ? min(token_pos[t], table_rows - 1) : 0;    // host-validated
        for (int c = lane; c < lay - kv_rank; c += 32)
            dst[kv_rank + c] = dl_from_f32<T>(lt_tail<T>(src + kv_rank, c, rot, rot_dims, cos_t, sin_t, pos));
    }
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const T* v = reinterpret_cast<const T*>(&raw[i]);
#pragma unroll
        for (int e = 0; e < V; ++e) { const float f = dl_to_f32<T>(v[e]); ss += f * f; }
    }
    const float r = 1.0f / sqrtf(dl_warp_sum(ss) / (float)rank + eps);
#pragma unroll
    for (int i = 0; i < NP; ++i) {
        const int c = (lane + 32 * i) * V;
        if (c >= rank) continue;
        T* v = reinterpret_cast<T*>(&raw[i]);
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] = dl_from_f32<T>(dl_to_f32<T>(v[e]) * r * (NP <= 4 ? gg[(i * V + e) % (NP <= 4 ? NP * V : 1)] : gain[c + e]));
        *reinterpret_cast<uint4*>(dst + c) = raw[i];
    }
}

// x [tokens, q_rank + kv_rank + rot] of dtype (rows ld apart; q_rank 0: no query latent); gains float32; cos, sin float32
// [table_rows, rot_dims / 2]; q_out [tokens, q_rank], kv_out [tokens, lay] contiguous of dtype, lay >= kv_rank + rot.
extern "C" int dl_latent_rows(const void* x, int dtype, int ld, int q_rank, int kv_rank, int rot, int rot_dims, const float* q_gain,
                              const float* kv_gain, float eps, const float* cos_t, const float* sin_t, int table_rows,
                              const int32_t* token_pos, void* q_out, void* kv_out, int lay, int n_tokens, void* stream) {
    DL_REQUIRE(n_tokens >= 0 && q_rank >= 0 && kv_rank > 0 && rot >= 0 && rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && eps > 0.f,
               "latent_rows: bad sizes");
    DL_REQUIRE(ld >= q_rank + kv_rank + rot && lay >= kv_rank + rot, "latent_rows: rows too short");
    DL_REQUIRE(dtype == DL_F32 || dtype == DL_BF16, "latent_rows: dtype %d", dtype);
    DL_REQUIRE(kv_gain && kv_out && (q_rank == 0 || (q_gain && q_out)) && (rot_dims == 0 || (cos_t && sin_t && token_pos && table_rows > 0)),
               "latent_rows: a tensor is missing");
    if (n_tokens == 0) return DL_OK;
    const dim3 grid(n_tokens, q_rank > 0 ? 2 : 1), block(LT_THREADS);
    const int v = dtype == DL_BF16 ? 8 : 4;
    const bool vec = q_rank % v == 0 && kv_rank % v == 0 && ld % v == 0 && lay % v == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)kv_out % 16) == 0 &&
                     ((uintptr_t)q_out % 16) == 0;
    cudaError_t e;
    const int longest = q_rank > kv_rank ? q_rank : kv_rank;
    if (vec && longest <= 32 * 8 * v && ((uintptr_t)q_gain % 16) == 0 && ((uintptr_t)kv_gain % 16) == 0) {
        const dim3 wgrid((n_tokens + LT_THREADS / 32 - 1) / (LT_THREADS / 32), grid.y);
#define LW_GO(T, NP)                                                                                                                       \
    e = dl_launch_dependent(latent_rows_warp_kernel<T, NP>, wgrid, block, 0, (cudaStream_t)stream, (const T*)x, ld, q_rank, kv_rank, rot,    \
                            rot_dims, q_gain, kv_gain, eps, cos_t, sin_t, table_rows, token_pos, (T*)q_out, (T*)kv_out, lay, n_tokens)
        if (dtype == DL_F32) { if (longest <= 32 * 4 * v) LW_GO(float, 4); else LW_GO(float, 8); }
        else { if (longest <= 32 * 4 * v) LW_GO(__nv_bfloat16, 4); else LW_GO(__nv_bfloat16, 8); }
#undef LW_GO
        if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "latent_rows: %s", cudaGetErrorString(e));
        return DL_OK;
    }
#define LR_GO(T, VEC)                                                                                                                    \
    e = dl_launch_dependent(latent_rows_kernel<T, VEC>, grid, block, 0, (cudaStream_t)stream, (const T*)x, ld, q_rank, kv_rank, rot, rot_dims, \
                            q_gain, kv_gain, eps, cos_t, sin_t, table_rows, token_pos, (T*)q_out, (T*)kv_out, lay)
    if (dtype == DL_F32 && vec) LR_GO(float, true);
    else if (dtype == DL_F32) LR_GO(float, false);
    else if (dtype == DL_BF16 && vec) LR_GO(__nv_bfloat16, true);
    else if (dtype == DL_BF16) LR_GO(__nv_bfloat16, false);
#undef LR_GO
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "latent_rows: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "latent_rows: %s", cudaGetErrorString(e));
    return DL_OK;
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_query_tail_kernel(const T* __restrict__ q, int q_ld, int dim, int rot, int rot_dims, const float* __restrict__ cos_t,
                         const float* __restrict__ sin_t, int table_rows, const int32_t* __restrict__ token_pos, T* __restrict__ out,
                         int out_ld, int rank, int lay, int H) {
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const size_t t = blockIdx.x;
    const int tail = lay - rank;
    const int pos = rot_dims > 0 ? min(token_pos[t], table_rows - 1) : 0;    // host-validated
    for (int e = threadIdx.x; e < H * tail; e += 256) {
        const int h = e / tail, c = e - h * tail;
        const T* src = q + t * q_ld + (size_t)h * (dim + rot) + dim;
        out[t * out_ld + (size_t)h * lay + rank + c] = dl_from_f32<T>(lt_tail<T>(src, c, rot, rot_dims, cos_t, sin_t, pos));
    }
}

// The same for bfloat16 tails that move 16 bytes at a time: a thread takes four pairs of one head.
__global__ void __launch_bounds__(256)
latent_query_tail_vec_kernel(const __nv_bfloat16* __restrict__ q, int q_ld, int dim, int rot, int rot_dims, const float* __restrict__ cos_t,
                             const float* __restrict__ sin_t, int table_rows, const int32_t* __restrict__ token_pos,
                             __nv_bfloat16* __restrict__ out, int out_ld, int rank, int lay, int H, int n_tokens) {
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const int units = (lay - rank) / 8, per_row = H * units;
    const long long idx = (long long)blockIdx.x * 256 + threadIdx.x;
    if (idx >= (long long)n_tokens * per_row) return;
    const int t = (int)(idx / per_row), e = (int)(idx - (long long)t * per_row), h = e / units, c = (e - h * units) * 8;
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
    if (c < rot) raw = *reinterpret_cast<const uint4*>(q + (size_t)t * q_ld + (size_t)h * (dim + rot) + dim + c);
    if (c < rot_dims) {
        const int pos = min(token_pos[t], table_rows - 1);       // host-validated
        const size_t at = (size_t)pos * (rot_dims / 2) + (c >> 1);
        const float4 cs = *reinterpret_cast<const float4*>(cos_t + at), sn = *reinterpret_cast<const float4*>(sin_t + at);
        const float cc[4] = {cs.x, cs.y, cs.z, cs.w}, ss[4] = {sn.x, sn.y, sn.z, sn.w};
        __nv_bfloat162* v = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            float a, b;
            lt_pair(__low2float(v[i]), __high2float(v[i]), cc[i], ss[i], a, b);
            v[i] = __floats2bfloat162_rn(a, b);
        }
    }
    *reinterpret_cast<uint4*>(out + (size_t)t * out_ld + (size_t)h * lay + rank + c) = raw;
}

extern "C" int dl_latent_query_tail(const void* q, int dtype, int q_ld, int dim, int rot, int rot_dims, const float* cos_t,
                                    const float* sin_t, int table_rows, const int32_t* token_pos, void* out, int out_ld, int rank,
                                    int lay, int H, int n_tokens, void* stream) {
    DL_REQUIRE(n_tokens >= 0 && H > 0 && dim >= 0 && rot >= 0 && rot_dims >= 0 && rot_dims <= rot && rot_dims % 2 == 0 && rank > 0,
               "latent_query_tail: bad sizes");
    DL_REQUIRE(q_ld >= H * (dim + rot) && lay >= rank + rot && out_ld >= H * lay, "latent_query_tail: rows too short");
    DL_REQUIRE(rot_dims == 0 || (cos_t && sin_t && token_pos && table_rows > 0), "latent_query_tail: a rotation needs tables and positions");
    if (n_tokens == 0 || lay == rank) return DL_OK;
    const dim3 grid(n_tokens), block(256);
    cudaError_t e;
    const uintptr_t places = (uintptr_t)q | (uintptr_t)out | (uintptr_t)cos_t | (uintptr_t)sin_t;
    if (dtype == DL_BF16 && places % 16 == 0 && q_ld % 8 == 0 && out_ld % 8 == 0 && dim % 8 == 0 && rot % 8 == 0 && rot_dims % 8 == 0 &&
        rank % 8 == 0 && lay % 8 == 0) {
        const long long n = (long long)n_tokens * H * ((lay - rank) / 8);
        e = dl_launch_dependent(latent_query_tail_vec_kernel, dim3((unsigned)((n + 255) / 256)), block, 0, (cudaStream_t)stream,
                                (const __nv_bfloat16*)q, q_ld, dim, rot, rot_dims, cos_t, sin_t, table_rows, token_pos,
                                (__nv_bfloat16*)out, out_ld, rank, lay, H, n_tokens);
        if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "latent_query_tail: %s", cudaGetErrorString(e));
        return DL_OK;
    }
    if (dtype == DL_F32)
        e = dl_launch_dependent(latent_query_tail_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)q, q_ld, dim, rot, rot_dims,
                                cos_t, sin_t, table_rows, token_pos, (float*)out, out_ld, rank, lay, H);
    else if (dtype == DL_BF16)
        e = dl_launch_dependent(latent_query_tail_kernel<__nv_bfloat16>, grid, block, 0, (cudaStream_t)stream, (const __nv_bfloat16*)q, q_ld,
                                dim, rot, rot_dims, cos_t, sin_t, table_rows, token_pos, (__nv_bfloat16*)out, out_ld, rank, lay, H);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "latent_query_tail: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "latent_query_tail: %s", cudaGetErrorString(e));
    return DL_OK;
}

// One block walks pieces of rows; VEC values (of one head) per thread at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
channel_gate_kernel(const T* __restrict__ o, int o_ld, int lay, const T* __restrict__ g, int g_ld, T* __restrict__ out, int out_ld,
                    int rows, int heads, int width, float scale) {
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const int per_row = heads * width / VEC;
    const size_t n = (size_t)rows * per_row;
    for (size_t i = (size_t)blockIdx.x * 256 + threadIdx.x; i < n; i += (size_t)gridDim.x * 256) {
        const size_t t = i / per_row;
        const int c = (int)(i - t * per_row) * VEC;
        const int h = c / width, d = c - h * width;
        const T* po = o + t * o_ld + (size_t)h * lay + d;
        const T* pg = g + t * g_ld + c;
        T* pd = out + t * out_ld + c;
        if (VEC == 1) {
            pd[0] = dl_from_f32<T>(g == nullptr ? scale * dl_to_f32<T>(po[0]) : scale * dl_to_f32<T>(po[0]) / (1.0f + expf(-dl_to_f32<T>(pg[0]))));
        } else {
            const uint4 ro = *reinterpret_cast<const uint4*>(po), rg = g == nullptr ? make_uint4(0u, 0u, 0u, 0u) : *reinterpret_cast<const uint4*>(pg);
            const T* vo = reinterpret_cast<const T*>(&ro);
            const T* vg = reinterpret_cast<const T*>(&rg);
            uint4 rd;
            T* vd = reinterpret_cast<T*>(&rd);
#pragma unroll
            for (int e = 0; e < VEC; ++e) vd[e] = dl_from_f32<T>(g == nullptr ? scale * dl_to_f32<T>(vo[e]) : scale * dl_to_f32<T>(vo[e]) / (1.0f + expf(-dl_to_f32<T>(vg[e]))));
            *reinterpret_cast<uint4*>(pd) = rd;
        }
    }
}

template <typename T>
static cudaError_t gate_launch(const void* o, int o_ld, int lay, const void* g, int g_ld, void* out, int out_ld, int rows, int heads,
                               int width, float scale, cudaStream_t s) {
    constexpr int V = 16 / sizeof(T);
    const bool vec = width % V == 0 && lay % V == 0 && o_ld % V == 0 && g_ld % V == 0 && out_ld % V == 0 && ((uintptr_t)o % 16) == 0 &&
                     ((uintptr_t)g % 16) == 0 && ((uintptr_t)out % 16) == 0;
    const size_t n = (size_t)rows * heads * width / (vec ? V : 1);
    const size_t want = (n + 255) / 256;
    const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16)), block(256);
    if (vec) return dl_launch_dependent(channel_gate_kernel<T, V>, grid, block, 0, s, (const T*)o, o_ld, lay, (const T*)g, g_ld, (T*)out, out_ld, rows, heads, width, scale);
    return dl_launch_dependent(channel_gate_kernel<T, 1>, grid, block, 0, s, (const T*)o, o_ld, lay, (const T*)g, g_ld, (T*)out, out_ld, rows, heads, width, scale);
}

// o [rows, heads * lay], g and out [rows, heads * width], all of dtype, rows o_ld / g_ld / out_ld apart.
extern "C" int dl_channel_gate(const void* o, int o_ld, int lay, const void* g, int g_ld, void* out, int out_ld, int dtype, int rows,
                               int heads, int width, float scale, void* stream) {
    DL_REQUIRE(rows >= 0 && heads > 0 && width > 0 && lay >= width && o_ld >= (heads - 1) * lay + width && g_ld >= heads * width &&
                   out_ld >= heads * width, "channel_gate: bad sizes");
    if (rows == 0) return DL_OK;
    cudaError_t e;
    if (dtype == DL_F32) e = gate_launch<float>(o, o_ld, lay, g, g_ld, out, out_ld, rows, heads, width, scale, (cudaStream_t)stream);
    else if (dtype == DL_BF16) e = gate_launch<__nv_bfloat16>(o, o_ld, lay, g, g_ld, out, out_ld, rows, heads, width, scale, (cudaStream_t)stream);
    else return dl_fail(DL_ERR_UNSUPPORTED, "channel_gate: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "channel_gate: %s", cudaGetErrorString(e));
    return DL_OK;
}

// ---------------------------------------------------------------------------------------------------------------------
// The change of basis per head for a few rows (a decode step), with what stands beside it in one kernel:
//
//   out[t, h * out_head + j] = f(sum_k W[h][j][k] x[t, h * x_head + k]),   f: nothing, or times sigmoid(gate[t, h * J + j])
//
// and, for queries on their way to the latent (`rot` >= 0), the rotated part of every head behind its J channels (rot channels of x
// behind its K, zeros up to out_head).  A warp owns 16 rows of W and 8 NT tokens: mma.sync m16n8k16 with W as A, the operands
// straight from memory, 16 bytes a lane (a lane's 8 neighbouring k of 32 are a permutation that both operands share).
#define PH_WARPS 2
#define PH_K 4                           // pieces of 32 channels whose operands are in flight together

__device__ __forceinline__ void ph_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <int NT>
__global__ void __launch_bounds__(32 * PH_WARPS)
per_head_rows_kernel(const __nv_bfloat16* __restrict__ x, int x_ld, int x_head, const __nv_bfloat16* __restrict__ w, int J, int K,
                     __nv_bfloat16* __restrict__ out, int out_ld, int out_head, const __nv_bfloat16* __restrict__ gate, int gate_ld, int rot,
                     int rot_dims, const float* __restrict__ cos_t, const float* __restrict__ sin_t, int table_rows,
                     const int32_t* __restrict__ token_pos, int n_tokens) {
    dl_launch_dependents();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
    const int h = blockIdx.y, tok0 = blockIdx.z * 8 * NT;
    const int j_lo = (blockIdx.x * PH_WARPS + warp) * 16 + g, j_hi = j_lo + 8;
    if (rot >= 0 && blockIdx.x == gridDim.x - 1) {           // a block of its own for what stands behind the J channels
        dl_grid_dependency_wait();
        const int tail = out_head - J, mine = min(8 * NT, n_tokens - tok0);
        for (int e = threadIdx.x; e < mine * tail; e += 32 * PH_WARPS) {
            const int tok = tok0 + e / tail, c = e % tail;
            const int pos = rot_dims > 0 ? min(token_pos[tok], table_rows - 1) : 0;       // host-validated
            out[(size_t)tok * out_ld + (size_t)h * out_head + J + c] = __float2bfloat16_rn(
                lt_tail<__nv_bfloat16>(x + (size_t)tok * x_ld + (size_t)h * x_head + K, c, rot, rot_dims, cos_t, sin_t, pos));
        }
        return;
    }
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    const __nv_bfloat16* w_lo = w + ((size_t)h * J + j_lo) * K + 8 * t;
    const __nv_bfloat16* w_hi = w_lo + (size_t)8 * K;
    // PH_K x 32 channels at a time: every operand of a run is asked for before the first product
    uint4 a_lo[PH_K], a_hi[PH_K];
    auto load_w = [&](int k0) {
#pragma unroll
        for (int i = 0; i < PH_K; ++i) {
            const bool in = k0 + 32 * i + 8 * t < K;
            a_lo[i] = in && j_lo < J ? *reinterpret_cast<const uint4*>(w_lo + k0 + 32 * i) : zero;
            a_hi[i] = in && j_hi < J ? *reinterpret_cast<const uint4*>(w_hi + k0 + 32 * i) : zero;
        }
    };
    load_w(0);                                               // weights: no kernel of the stream writes them
    dl_grid_dependency_wait();
    float acc[NT][4], gv[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int tok = tok0 + 8 * n + 2 * t + (e & 1), j = e < 2 ? j_lo : j_hi;
            acc[n][e] = 0.f;
            gv[n][e] = gate != nullptr && tok < n_tokens && j < J ? __bfloat162float(gate[(size_t)tok * gate_ld + (size_t)h * J + j]) : 0.f;
        }
    for (int k0 = 0; k0 < K; k0 += 32 * PH_K) {
        uint4 b[NT][PH_K];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int i = 0; i < PH_K; ++i) {
                const int tok = tok0 + 8 * n + g, k = k0 + 32 * i + 8 * t;
                b[n][i] = tok < n_tokens && k < K ? *reinterpret_cast<const uint4*>(x + (size_t)tok * x_ld + (size_t)h * x_head + k) : zero;
            }
        if (k0 > 0) load_w(k0);
#pragma unroll
        for (int i = 0; i < PH_K; ++i)
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                ph_mma(acc[n], a_lo[i].x, a_hi[i].x, a_lo[i].y, a_hi[i].y, b[n][i].x, b[n][i].y);
                ph_mma(acc[n], a_lo[i].z, a_hi[i].z, a_lo[i].w, a_hi[i].w, b[n][i].z, b[n][i].w);
            }
    }
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int tok = tok0 + 8 * n + 2 * t + (e & 1), j = e < 2 ? j_lo : j_hi;
            if (tok >= n_tokens || j >= J) continue;
            const float v = gate != nullptr ? acc[n][e] / (1.0f + expf(-gv[n][e])) : acc[n][e];
            out[(size_t)tok * out_ld + (size_t)h * out_head + j] = __float2bfloat16_rn(v);
        }
}

// x bf16 [tokens, H * x_head] (rows x_ld apart), w bf16 [H, J, K], out bf16 [tokens, H * out_head] (rows out_ld apart); K, x_ld and
// x_head multiples of 8, x and w 16-byte aligned.  gate bf16 [tokens, H * J] (rows gate_ld apart) or NULL; rot -1: nothing behind the
// J channels, else as in dl_latent_query_tail.
extern "C" int dl_per_head_rows(const void* x, int x_ld, int x_head, const void* w, int H, int J, int K, void* out, int out_ld, int out_head,
                                const void* gate, int gate_ld, int rot, int rot_dims, const float* cos_t, const float* sin_t, int table_rows,
                                const int32_t* token_pos, int n_tokens, void* stream) {
    DL_REQUIRE(n_tokens >= 0 && H > 0 && J > 0 && K > 0 && H <= 65535, "per_head_rows: bad sizes");
    DL_REQUIRE(K % 8 == 0 && x_ld % 8 == 0 && x_head % 8 == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)w % 16) == 0, "per_head_rows: operands come in aligned eights");
    DL_REQUIRE(x_head >= K + (rot > 0 ? rot : 0) && out_head >= J + (rot > 0 ? rot : 0) && x_ld >= H * x_head && out_ld >= H * out_head &&
                   (gate == nullptr || gate_ld >= H * J), "per_head_rows: rows overlap");
    DL_REQUIRE(rot_dims >= 0 && rot_dims <= (rot > 0 ? rot : 0) && rot_dims % 2 == 0 && (rot_dims == 0 || (cos_t && sin_t && token_pos && table_rows > 0)),
               "per_head_rows: a rotation needs tables and positions");
    if (n_tokens == 0) return DL_OK;
    const int nt = n_tokens <= 8 ? 1 : 2;
    const dim3 grid((J + 16 * PH_WARPS - 1) / (16 * PH_WARPS) + (rot >= 0 ? 1 : 0), H, (n_tokens + 8 * nt - 1) / (8 * nt)), block(32 * PH_WARPS);
    cudaError_t e;
#define PH_GO(NT)                                                                                                                          \
    e = dl_launch_dependent(per_head_rows_kernel<NT>, grid, block, 0, (cudaStream_t)stream, (const __nv_bfloat16*)x, x_ld, x_head,         \
                            (const __nv_bfloat16*)w, J, K, (__nv_bfloat16*)out, out_ld, out_head, (const __nv_bfloat16*)gate, gate_ld, rot, \
                            rot_dims, cos_t, sin_t, table_rows, token_pos, n_tokens)
    if (nt == 1) PH_GO(1);
    else PH_GO(2);
#undef PH_GO
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "per_head_rows: %s", cudaGetErrorString(e));
    return DL_OK;
}
