// Row gather: token embedding lookup into the float32 residual stream, and selection of
// the rows whose logits are wanted.
//
// Role of the reference's embedding_lookup_* kernels (native/kernels/embedding.cu:30-46,
// native/kernels/embedding_f32out.cu:10-70): one block per output row, the row copied
// with widening to float32 (or kept in bfloat16, for rows of activations that go on to a product).
#include "common.cuh"

template <typename T, typename TOut>
__global__ void __launch_bounds__(256)
gather_rows_kernel(const T* __restrict__ table, int table_stride, const int32_t* __restrict__ ids,
                   TOut* __restrict__ out, int width, int n_table_rows) {
    dl_launch_dependents();
    const int row = blockIdx.x;
    const int id = ids[row];
    TOut* dst = out + (size_t)row * width;
    if (id < 0 || id >= n_table_rows) {          // the host validates ids; never read outside the table
        for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = dl_from_f32<TOut>(0.f);
        return;
    }
    const T* src = table + (size_t)id * table_stride;
    for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = dl_from_f32<TOut>(dl_to_f32<T>(src[c]));
}

// out[r, :] = table[ids[r], :] as `out_dtype`.  table: [n_table_rows, width] of `dtype`, rows
// table_stride elements apart; out: contiguous [n_rows, width], float32 or (from a bfloat16 table) bfloat16.
extern "C" int dl_gather_rows(const void* table, int dtype, int table_stride, const int32_t* ids, void* out, int out_dtype,
                              int n_rows, int width, int n_table_rows, void* stream) {
    DL_REQUIRE(n_rows >= 0 && width > 0 && n_table_rows > 0 && table_stride >= width,
               "gather_rows: bad sizes rows=%d width=%d table=%d stride=%d", n_rows, width, n_table_rows, table_stride);
    if (n_rows == 0) return DL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == DL_F32 && out_dtype == DL_F32)
        gather_rows_kernel<float, float><<<n_rows, 256, 0, s>>>((const float*)table, table_stride, ids, (float*)out, width, n_table_rows);
    else if (dtype == DL_BF16 && out_dtype == DL_F32)
        gather_rows_kernel<__nv_bfloat16, float><<<n_rows, 256, 0, s>>>((const __nv_bfloat16*)table, table_stride, ids, (float*)out,
                                                                         width, n_table_rows);
    else if (dtype == DL_BF16 && out_dtype == DL_BF16)
        gather_rows_kernel<__nv_bfloat16, __nv_bfloat16><<<n_rows, 256, 0, s>>>((const __nv_bfloat16*)table, table_stride, ids,
                                                                                 (__nv_bfloat16*)out, width, n_table_rows);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "gather_rows: from dtype %d to dtype %d", dtype, out_dtype);
    DL_CHECK_LAUNCH("gather_rows");
    return DL_OK;
}

// Token embedding plus a learned position vector: out[r, :] = table[ids[r], :] + positions[pos[r], :],
// the sum in float32.  One block per row.
template <typename T>
__global__ void __launch_bounds__(256)
embed_positions_kernel(const T* __restrict__ table, const T* __restrict__ pos_table, const int32_t* __restrict__ ids,
                       const int32_t* __restrict__ pos, float* __restrict__ out, int width, int n_table_rows,
                       int n_positions) {
    dl_launch_dependents();
    const int row = blockIdx.x;
    const int id = ids[row], p = pos[row];
    float* dst = out + (size_t)row * width;
    const bool ok = id >= 0 && id < n_table_rows && p >= 0 && p < n_positions;   // host-validated
    const T* a = table + (size_t)(ok ? id : 0) * width;
    const T* b = pos_table + (size_t)(ok ? p : 0) * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x) dst[c] = ok ? dl_to_f32<T>(a[c]) + dl_to_f32<T>(b[c]) : 0.f;
}

// table [n_table_rows, width], pos_table [n_positions, width] of `dtype`, both contiguous; out float32 [n_rows, width].
extern "C" int dl_embed_positions(const void* table, const void* pos_table, int dtype, const int32_t* ids,
                                  const int32_t* pos, float* out, int n_rows, int width, int n_table_rows,
                                  int n_positions, void* stream) {
    DL_REQUIRE(n_rows >= 0 && width > 0 && n_table_rows > 0 && n_positions > 0, "embed_positions: bad sizes");
    if (n_rows == 0) return DL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == DL_F32)
        embed_positions_kernel<float><<<n_rows, 256, 0, s>>>((const float*)table, (const float*)pos_table, ids, pos, out, width,
                                                             n_table_rows, n_positions);
    else if (dtype == DL_BF16)
        embed_positions_kernel<__nv_bfloat16><<<n_rows, 256, 0, s>>>((const __nv_bfloat16*)table, (const __nv_bfloat16*)pos_table,
                                                                     ids, pos, out, width, n_table_rows, n_positions);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "embed_positions: dtype %d", dtype);
    DL_CHECK_LAUNCH("embed_positions");
    return DL_OK;
}

// Token embedding times a constant plus a row of a table of token pairs:
//   out[r, :] = table[ids[r], :] * scale + pairs[(before * mul_prev + ids[r] * mul_cur) mod buckets, :]
// with `before` the token ahead of ids[r] in its sequence; a sequence's first token takes row `buckets`, the last.  Inside a
// step the token ahead is the packed row ahead; for the first of a sequence's new tokens it is what the sequence's slot of
// `last` holds, which then becomes the last of the new ones (one block reads and writes it).  The sum in float32.  One block
// per row, VEC values a thread at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256)
embed_pairs_kernel(const T* __restrict__ table, const T* __restrict__ pairs, const int32_t* __restrict__ ids,
                   const int32_t* __restrict__ token_seq, const int32_t* __restrict__ token_pos, const int32_t* __restrict__ cu_new,
                   const int32_t* __restrict__ slots, int32_t* __restrict__ last, int last_stride, int n_slots, float* __restrict__ out,
                   int width, int n_table_rows, int buckets, long long mul_prev, long long mul_cur, float scale) {
    __shared__ int s_pair;
    dl_launch_dependents();
    const int row = blockIdx.x;
    const int id = ids[row];
    if (threadIdx.x == 0) {
        const int seq = token_seq[row], first = cu_new[seq];
        long long before = -1;
        if (row != first) {
            before = ids[row - 1];
        } else {
            const int slot = slots[seq];
            if (slot >= 0 && slot < n_slots) {               // host-validated
                int32_t* mine = last + (size_t)slot * last_stride;
                if (token_pos[row] > 0) before = *mine;
                *mine = ids[cu_new[seq + 1] - 1];
            }
        }
        long long pair = buckets;
        if (before >= 0) {
            pair = (before * mul_prev + (long long)id * mul_cur) % buckets;
            if (pair < 0) pair += buckets;
        }
        s_pair = (int)pair;
    }
    __syncthreads();
    const bool ok = id >= 0 && id < n_table_rows;            // host-validated; never read outside the table
    const T* a = table + (size_t)(ok ? id : 0) * width;
    const T* b = pairs + (size_t)s_pair * width;
    float* dst = out + (size_t)row * width;
    for (int c = threadIdx.x * VEC; c < width; c += 256 * VEC) {
        if constexpr (VEC == 1) {
            dst[c] = ok ? dl_to_f32<T>(a[c]) * scale + dl_to_f32<T>(b[c]) : 0.f;
        } else {
            constexpr int W = VEC * (int)sizeof(T) / 8;      // pieces of 8 bytes
            uint2 ra[W], rb[W];
#pragma unroll
            for (int i = 0; i < W; ++i) {
                ra[i] = *(reinterpret_cast<const uint2*>(a + c) + i);
                rb[i] = *(reinterpret_cast<const uint2*>(b + c) + i);
            }
            const T* va = reinterpret_cast<const T*>(ra);
            const T* vb = reinterpret_cast<const T*>(rb);
            float v[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) v[e] = ok ? dl_to_f32<T>(va[e]) * scale + dl_to_f32<T>(vb[e]) : 0.f;
#pragma unroll
            for (int e = 0; e < VEC; e += 4) *reinterpret_cast<float4*>(dst + c + e) = make_float4(v[e], v[e + 1], v[e + 2], v[e + 3]);
        }
    }
}

// table [n_table_rows, width], pairs [buckets + 1, width] of `dtype`, contiguous; ids, token_seq, token_pos int32 [n_rows];
// cu_new int32 [sequences + 1], slots int32 [sequences]; last: int32, one value per slot, last_stride apart; out float32
// [n_rows, width].
extern "C" int dl_embed_pairs(const void* table, const void* pairs, int dtype, const int32_t* ids, const int32_t* token_seq,
                              const int32_t* token_pos, const int32_t* cu_new, const int32_t* slots, int32_t* last, int last_stride,
                              int n_slots, float* out, int n_rows, int width, int n_table_rows, int buckets, long long mul_prev,
                              long long mul_cur, float scale, void* stream) {
    DL_REQUIRE(n_rows >= 0 && width > 0 && n_table_rows > 0 && buckets > 0 && last_stride > 0 && n_slots > 0, "embed_pairs: bad sizes");
    DL_REQUIRE(table && pairs && ids && token_seq && token_pos && cu_new && slots && last && out, "embed_pairs: a tensor is missing");
    DL_REQUIRE(dtype == DL_F32 || dtype == DL_BF16, "embed_pairs: dtype %d", dtype);
    if (n_rows == 0) return DL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && (((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)out) % 16) == 0;
#define EP_GO(T, VEC)                                                                                                                   \
    embed_pairs_kernel<T, VEC><<<n_rows, 256, 0, s>>>((const T*)table, (const T*)pairs, ids, token_seq, token_pos, cu_new, slots, last,  \
                                                      last_stride, n_slots, out, width, n_table_rows, buckets, mul_prev, mul_cur, scale)
    if (dtype == DL_F32) { if (vec) EP_GO(float, 4); else EP_GO(float, 1); }
    else { if (vec) EP_GO(__nv_bfloat16, 4); else EP_GO(__nv_bfloat16, 1); }
#undef EP_GO
    DL_CHECK_LAUNCH("embed_pairs");
    return DL_OK;
}
