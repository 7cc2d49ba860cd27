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

#define LT_THREADS 128

template <typename T>
__global__ void __launch_bounds__(LT_THREADS)
latent_rows_kernel(const T* __restrict__ x, int ld, int q_rank, int kv_rank, int rot, int rot_dims, const float* __restrict__ q_gain,
                   const float* __restrict__ kv_gain, float eps, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                   int table_rows, const int32_t* __restrict__ token_pos, T* __restrict__ q_out, T* __restrict__ kv_out, int lay) {
    __shared__ float scratch[33];
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const size_t t = blockIdx.x;
    const bool is_q = blockIdx.y == 1;
    const int rank = is_q ? q_rank : kv_rank;
    const T* src = x + t * ld + (is_q ? 0 : q_rank);
    T* dst = is_q ? q_out + t * q_rank : kv_out + t * lay;
    const float* gain = is_q ? q_gain : kv_gain;
    float ss = 0.f;
    for (int c = threadIdx.x; c < rank; c += LT_THREADS) { const float v = dl_to_f32<T>(src[c]); ss += v * v; }
    ss = dl_block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)rank + eps);
    for (int c = threadIdx.x; c < rank; c += LT_THREADS) dst[c] = dl_from_f32<T>(dl_to_f32<T>(src[c]) * r * gain[c]);
    if (is_q) return;
    const int pos = rot_dims > 0 ? min(token_pos[t], table_rows - 1) : 0;    // host-validated
    for (int c = threadIdx.x; c < lay - kv_rank; c += LT_THREADS) {
        float v = c < rot ? dl_to_f32<T>(src[kv_rank + c]) : 0.f;
        if (c < rot_dims) {
            const int i = c >> 1;
            const float other = dl_to_f32<T>(src[kv_rank + (c ^ 1)]);
            const float cs = cos_t[(size_t)pos * (rot_dims / 2) + i], sn = sin_t[(size_t)pos * (rot_dims / 2) + i];
            float a, b;
            lt_pair(c & 1 ? other : v, c & 1 ? v : other, cs, sn, a, b);
            v = c & 1 ? b : a;
        }
        dst[kv_rank + c] = dl_from_f32<T>(v);
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
    DL_REQUIRE(kv_gain && kv_out && (q_rank == 0 || (q_gain && q_out)) && (rot_dims == 0 || (cos_t && sin_t && token_pos && table_rows > 0)),
               "latent_rows: a tensor is missing");
    if (n_tokens == 0) return DL_OK;
    const dim3 grid(n_tokens, q_rank > 0 ? 2 : 1), block(LT_THREADS);
    cudaError_t e;
    if (dtype == DL_F32)
        e = dl_launch_dependent(latent_rows_kernel<float>, grid, block, 0, (cudaStream_t)stream, (const float*)x, ld, q_rank, kv_rank, rot,
                                rot_dims, q_gain, kv_gain, eps, cos_t, sin_t, table_rows, token_pos, (float*)q_out, (float*)kv_out, lay);
    else if (dtype == DL_BF16)
        e = dl_launch_dependent(latent_rows_kernel<__nv_bfloat16>, grid, block, 0, (cudaStream_t)stream, (const __nv_bfloat16*)x, ld, q_rank,
                                kv_rank, rot, rot_dims, q_gain, kv_gain, eps, cos_t, sin_t, table_rows, token_pos, (__nv_bfloat16*)q_out,
                                (__nv_bfloat16*)kv_out, lay);
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
        float v = c < rot ? dl_to_f32<T>(src[c]) : 0.f;
        if (c < rot_dims) {
            const int i = c >> 1;
            const float other = dl_to_f32<T>(src[c ^ 1]);
            const float cs = cos_t[(size_t)pos * (rot_dims / 2) + i], sn = sin_t[(size_t)pos * (rot_dims / 2) + i];
            float a, b;
            lt_pair(c & 1 ? other : v, c & 1 ? v : other, cs, sn, a, b);
            v = c & 1 ? b : a;
        }
        out[t * out_ld + (size_t)h * lay + rank + c] = dl_from_f32<T>(v);
    }
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
