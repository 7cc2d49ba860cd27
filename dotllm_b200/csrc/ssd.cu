// A state-space recurrence with one decay per head and token (the state-space dual form of Mamba-2):
//
//   dt_t = softplus(z_t + dt_bias_h)
//   S_t  = exp(-exp(A_h) dt_t) S_(t-1) + dt_t B_t x_t^T          (S: [state channels, value channels] per head)
//   y_t  = S_t^T C_t + D_h x_t
//
// heads / groups neighbouring heads share a group's B and C.  Everything here is float32: the inputs come from a short
// convolution in float32 (csrc/causal_conv.cu), only the step logits z are read in the projection's type.
//
// The scan walks a sequence's new tokens in order from the slot's state and leaves the new state there: a prompt, a part of a
// prompt and one decoded token are the same loop, so a position's result does not depend on how its sequence was cut into
// steps.  A block owns COLS value channels of one (sequence, head); columns of S never mix.  A thread holds a tile of ROWS
// state channels x CPT value channels in registers, so that the eight operands B and C it reads from shared memory serve
// CPT columns each; SS_SPLIT threads share a column.  Tokens are staged a batch at a time from registers that were loaded
// while the batch before was walked.  Nothing in the walk waits for another lane: a thread leaves its share of y in shared
// memory and the shares of a batch are summed afterwards, in a fixed order.
#include "common.cuh"

#define SS_SPLIT 16                      // threads that share a column
#define SS_GROUPS 8                      // column groups of a block
#define SS_THREADS (SS_SPLIT * SS_GROUPS)
#define SS_MAX_STATE 512
#define SS_STAGE 1024                    // values of B (and of C) staged per batch
#define SS_MAX_BATCH 8

__device__ __forceinline__ float ss_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }

template <typename T, int ROWS, int CPT, bool SINGLE>
__global__ void __launch_bounds__(SS_THREADS)
ssd_scan_kernel(const float* __restrict__ xbc, int ld, const T* __restrict__ z, int z_ld, const float* __restrict__ dt_bias,
                const float* __restrict__ a_log, const float* __restrict__ skip, const int32_t* __restrict__ cu_new,
                const int32_t* __restrict__ slots, float* __restrict__ state, long slot_stride, int n_slots,
                float* __restrict__ y, int y_ld, int H, int G, int N, int P, int vec_state) {
    constexpr int COLS = SS_GROUPS * CPT;
    constexpr int PAD = SS_SPLIT * ROWS;                       // staged state channels per token, >= N
    constexpr int BATCH = SINGLE ? 1 : (SS_STAGE / PAD < SS_MAX_BATCH ? SS_STAGE / PAD : SS_MAX_BATCH);
    constexpr int LOADS = (BATCH * PAD + SS_THREADS - 1) / SS_THREADS;
    constexpr int XLOADS = (BATCH * COLS + SS_THREADS - 1) / SS_THREADS;
    __shared__ __align__(16) float sB[2][BATCH * PAD], sC[2][BATCH * PAD];
    __shared__ __align__(16) float sx[2][XLOADS * SS_THREADS];
    __shared__ float sa[2][BATCH], sdt[2][BATCH];
    __shared__ __align__(16) float sp[BATCH * SS_SPLIT * COLS];  // every thread's share of y, [token][share][column]
    dl_launch_dependents();
    const int b = blockIdx.z, h = blockIdx.y, g = h / (H / G);
    const int tid = threadIdx.x, r = tid / SS_GROUPS, cg = tid % SS_GROUPS;
    const int col0 = blockIdx.x * COLS, col = col0 + cg * CPT;
    const float rate = expf(a_log[h]), bias = dt_bias[h], d_skip = skip[h];
    dl_grid_dependency_wait();
    const int t0 = cu_new[b], t1 = cu_new[b + 1];
    const int slot = slots[b];
    if (slot < 0 || slot >= n_slots || t0 >= t1) return;      // uniform over the block
    float* S = state + (size_t)slot * slot_stride + (size_t)h * N * P;
    float s[ROWS][CPT];
#pragma unroll
    for (int m = 0; m < ROWS; ++m) {
        const int ch = r * ROWS + m;
        if (CPT == 4 && vec_state) {                           // P a multiple of 4 and rows 16-byte aligned
            const float4 v = ch < N && col < P ? *reinterpret_cast<const float4*>(S + (size_t)ch * P + col) : make_float4(0.f, 0.f, 0.f, 0.f);
            s[m][0] = v.x, s[m][1 % CPT] = v.y, s[m][2 % CPT] = v.z, s[m][3 % CPT] = v.w;
        } else {
#pragma unroll
            for (int e = 0; e < CPT; ++e) s[m][e] = ch < N && col + e < P ? S[(size_t)ch * P + col + e] : 0.f;
        }
    }
    const float* x_in = xbc + (size_t)h * P;
    const float* b_in = xbc + (size_t)H * P + (size_t)g * N;
    const float* c_in = b_in + (size_t)G * N;
    float rB[LOADS], rC[LOADS], rx[XLOADS], rz = 0.f;
    auto fetch = [&](int first, int count) {                   // every load from a valid (clamped) address; what lies outside is dropped when staged
#pragma unroll
        for (int l = 0; l < LOADS; ++l) {
            const int e = tid + SS_THREADS * l;
            const size_t row = (size_t)(first + min(e / PAD, count - 1)) * ld;
            const int ch = min(e % PAD, N - 1);
            rB[l] = b_in[row + ch];
            rC[l] = c_in[row + ch];
        }
#pragma unroll
        for (int l = 0; l < XLOADS; ++l) {
            const int e = tid + SS_THREADS * l;
            rx[l] = x_in[(size_t)(first + min(e / COLS, count - 1)) * ld + min(col0 + e % COLS, P - 1)];
        }
        rz = dl_to_f32<T>(z[(size_t)(first + min(tid, count - 1)) * z_ld + h]);
    };
    fetch(t0, min(BATCH, t1 - t0));
    int buf = 0;
    for (int first = t0; first < t1; first += BATCH) {
        const int count = min(BATCH, t1 - first);
#pragma unroll
        for (int l = 0; l < LOADS; ++l) {
            const int e = tid + SS_THREADS * l;
            if (e < BATCH * PAD) {
                const bool live = e / PAD < count && e % PAD < N;   // a padded channel holds zeros and stays zero
                sB[buf][e] = live ? rB[l] : 0.f;
                sC[buf][e] = live ? rC[l] : 0.f;
            }
        }
#pragma unroll
        for (int l = 0; l < XLOADS; ++l) sx[buf][tid + SS_THREADS * l] = rx[l];
        if (tid < BATCH) {
            const float dt = ss_softplus(rz + bias);
            sdt[buf][tid] = dt;
            sa[buf][tid] = expf(-rate * dt);
        }
        __syncthreads();                                        // the batch is staged; the shares of the batch before are summed
        if (first + BATCH < t1) fetch(first + BATCH, min(BATCH, t1 - first - BATCH));
#pragma unroll 2
        for (int i = 0; i < count; ++i) {
            const float a = sa[buf][i], dt = sdt[buf][i];
            float xv[CPT], o[CPT];
#pragma unroll
            for (int e = 0; e < CPT; ++e) xv[e] = sx[buf][i * COLS + cg * CPT + e] * dt, o[e] = 0.f;
            float bb[ROWS], cc[ROWS];
            if (ROWS % 4 == 0) {
                const float4* pb = reinterpret_cast<const float4*>(sB[buf] + i * PAD + r * ROWS);
                const float4* pc = reinterpret_cast<const float4*>(sC[buf] + i * PAD + r * ROWS);
#pragma unroll
                for (int m = 0; m < ROWS / 4; ++m) {
                    const float4 b4 = pb[m], c4 = pc[m];
                    bb[4 * m] = b4.x, bb[(4 * m + 1) % ROWS] = b4.y, bb[(4 * m + 2) % ROWS] = b4.z, bb[(4 * m + 3) % ROWS] = b4.w;
                    cc[4 * m] = c4.x, cc[(4 * m + 1) % ROWS] = c4.y, cc[(4 * m + 2) % ROWS] = c4.z, cc[(4 * m + 3) % ROWS] = c4.w;
                }
            } else {
#pragma unroll
                for (int m = 0; m < ROWS; ++m) bb[m] = sB[buf][i * PAD + r * ROWS + m], cc[m] = sC[buf][i * PAD + r * ROWS + m];
            }
#pragma unroll
            for (int m = 0; m < ROWS; ++m)
#pragma unroll
                for (int e = 0; e < CPT; ++e) {
                    s[m][e] = fmaf(a, s[m][e], bb[m] * xv[e]);
                    o[e] = fmaf(s[m][e], cc[m], o[e]);
                }
            float* share = sp + (i * SS_SPLIT + r) * COLS + cg * CPT;
            if (CPT == 4) {
                *reinterpret_cast<float4*>(share) = make_float4(o[0], o[1 % CPT], o[2 % CPT], o[3 % CPT]);
            } else {
#pragma unroll
                for (int e = 0; e < CPT; ++e) share[e] = o[e];
            }
        }
        __syncthreads();
        for (int e = tid; e < count * COLS; e += SS_THREADS) {
            const float* part = sp + (e / COLS) * SS_SPLIT * COLS + e % COLS;
            float total = 0.f;
#pragma unroll
            for (int p4 = 0; p4 < SS_SPLIT; p4 += 4)
                total += (part[p4 * COLS] + part[(p4 + 1) * COLS]) + (part[(p4 + 2) * COLS] + part[(p4 + 3) * COLS]);
            const int c = col0 + e % COLS;
            if (c < P) y[(size_t)(first + e / COLS) * y_ld + h * P + c] = fmaf(d_skip, sx[buf][e], total);
        }
        buf ^= 1;
    }
#pragma unroll
    for (int m = 0; m < ROWS; ++m) {
        const int ch = r * ROWS + m;
        if (ch >= N) continue;
        if (CPT == 4 && vec_state) {
            if (col < P) *reinterpret_cast<float4*>(S + (size_t)ch * P + col) = make_float4(s[m][0], s[m][1 % CPT], s[m][2 % CPT], s[m][3 % CPT]);
        } else {
#pragma unroll
            for (int e = 0; e < CPT; ++e)
                if (col + e < P) S[(size_t)ch * P + col + e] = s[m][e];
        }
    }
}

template <typename T>
static cudaError_t ssd_launch(const float* xbc, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log,
                              const float* skip, const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride,
                              int n_slots, float* y, int y_ld, int n_seqs, int n_tokens, int H, int G, int N, int P, cudaStream_t s) {
    const bool single = n_tokens == n_seqs;                   // every sequence brings exactly one token
    const int vec_state = P % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state % 16) == 0;
    const int rows = (N + SS_SPLIT - 1) / SS_SPLIT;
#define SS_GO(ROWS, CPT)                                                                                                      \
    do {                                                                                                                      \
        const dim3 grid((P + SS_GROUPS * CPT - 1) / (SS_GROUPS * CPT), H, n_seqs), block(SS_THREADS);                        \
        /* few blocks that walk a long run of tokens want a multiprocessor each */                                            \
        const bool early = (long)grid.x * grid.y * grid.z > 2L * dl_sm_count();                                              \
        if (single)                                                                                                           \
            return dl_launch_dependent_if(early, ssd_scan_kernel<T, ROWS, CPT, true>, grid, block, 0, s, xbc, ld, (const T*)z, \
                                          z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, H, \
                                          G, N, P, vec_state);                                                                \
        return dl_launch_dependent_if(early, ssd_scan_kernel<T, ROWS, CPT, false>, grid, block, 0, s, xbc, ld, (const T*)z,   \
                                      z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, H, G,  \
                                      N, P, vec_state);                                                                       \
    } while (0)
    if (rows <= 1) SS_GO(1, 4);
    if (rows <= 2) SS_GO(2, 4);
    if (rows <= 4) SS_GO(4, 4);
    if (rows <= 8) SS_GO(8, 4);
    if (rows <= 16) SS_GO(16, 2);
    SS_GO(32, 1);
#undef SS_GO
}

// xbc float32 [tokens, H*P + 2*G*N] (rows ld apart): x, then B, then C; z [tokens, H] of z_dtype (rows z_ld apart): the step
// logits; dt_bias, a_log, skip float32 [H]; state float32 [N, P] per head at `state` + slot * slot_stride; y float32 [tokens, H*P].
extern "C" int dl_ssd_scan(const float* xbc, int ld, const void* z, int z_dtype, int z_ld, const float* dt_bias, const float* a_log,
                           const float* skip, const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride,
                           int n_slots, float* y, int y_ld, int n_seqs, int n_tokens, int H, int G, int N, int P, void* stream) {
    DL_REQUIRE(n_seqs >= 0 && n_tokens >= 0 && H > 0 && G > 0 && N > 0 && P > 0 && n_slots > 0 && H % G == 0, "ssd_scan: bad sizes");
    DL_REQUIRE(N <= SS_MAX_STATE, "ssd_scan: a state of %d channels, the kernel takes up to %d", N, SS_MAX_STATE);
    DL_REQUIRE(ld >= H * P + 2 * G * N && z_ld >= H && y_ld >= H * P && slot_stride >= (long)H * N * P, "ssd_scan: rows overlap");
    DL_REQUIRE(H <= 65535 && n_seqs <= 65535, "ssd_scan: too many heads or sequences");
    if (n_seqs == 0 || n_tokens == 0) return DL_OK;
    cudaError_t e;
    if (z_dtype == DL_F32)
        e = ssd_launch<float>(xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, n_seqs, n_tokens, H, G, N, P, (cudaStream_t)stream);
    else if (z_dtype == DL_BF16)
        e = ssd_launch<__nv_bfloat16>(xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, n_seqs, n_tokens, H, G, N, P, (cudaStream_t)stream);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "ssd_scan: dtype %d", z_dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "ssd_scan: %s", cudaGetErrorString(e));
    return DL_OK;
}

// A gate in front of a norm over equal parts of a row:
//   v = y * silu(g);  out = scale * v / sqrt(mean over the part of v^2 + eps) * gain
// One block per (row, part).  y float32, g of the step's type, float32 arithmetic; rows of g and out may be column views.
#define GN_THREADS 256
#define GN_KEEP 16                       // values a thread keeps in registers; wider parts are computed twice

template <typename T>
__global__ void __launch_bounds__(GN_THREADS)
gated_group_norm_kernel(const float* __restrict__ y, int y_ld, const T* __restrict__ g, int g_ld, const float* __restrict__ gain,
                        T* __restrict__ out, int out_ld, int part, float eps, float scale) {
    __shared__ float scratch[33];
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const int c0 = blockIdx.y * part;
    const float* yr = y + (size_t)blockIdx.x * y_ld + c0;
    const T* gr = g + (size_t)blockIdx.x * g_ld + c0;
    T* dst = out + (size_t)blockIdx.x * out_ld + c0;
    auto value = [&](int c) {
        const float gate = dl_to_f32<T>(gr[c]);
        return yr[c] * (gate / (1.0f + expf(-gate)));
    };
    float v[GN_KEEP];
    float ss = 0.f;
    const bool keep = part <= GN_THREADS * GN_KEEP;
    if (keep) {
#pragma unroll
        for (int i = 0; i < GN_KEEP; ++i) {
            const int c = threadIdx.x + i * GN_THREADS;
            v[i] = c < part ? value(c) : 0.f;
            ss += v[i] * v[i];
        }
    } else {
        for (int c = threadIdx.x; c < part; c += GN_THREADS) { const float w = value(c); ss += w * w; }
    }
    ss = dl_block_sum(ss, scratch);
    const float r = scale / sqrtf(ss / (float)part + eps);
    if (keep) {
#pragma unroll
        for (int i = 0; i < GN_KEEP; ++i) {
            const int c = threadIdx.x + i * GN_THREADS;
            if (c < part) dst[c] = dl_from_f32<T>(v[i] * r * gain[c0 + c]);
        }
    } else {
        for (int c = threadIdx.x; c < part; c += GN_THREADS) dst[c] = dl_from_f32<T>(value(c) * r * gain[c0 + c]);
    }
}

extern "C" int dl_gated_group_norm(const float* y, int y_ld, const void* g, int g_ld, const float* gain, void* out, int out_ld,
                                   int dtype, int rows, int width, int parts, float eps, float scale, void* stream) {
    DL_REQUIRE(rows >= 0 && width > 0 && parts > 0 && width % parts == 0 && parts <= 65535 && eps > 0.f, "gated_group_norm: bad sizes");
    DL_REQUIRE(y_ld >= width && g_ld >= width && out_ld >= width, "gated_group_norm: rows overlap");
    if (rows == 0) return DL_OK;
    const dim3 grid(rows, parts), block(GN_THREADS);
    cudaError_t e;
    if (dtype == DL_F32)
        e = dl_launch_dependent(gated_group_norm_kernel<float>, grid, block, 0, (cudaStream_t)stream, y, y_ld, (const float*)g, g_ld, gain,
                                (float*)out, out_ld, width / parts, eps, scale);
    else if (dtype == DL_BF16)
        e = dl_launch_dependent(gated_group_norm_kernel<__nv_bfloat16>, grid, block, 0, (cudaStream_t)stream, y, y_ld,
                                (const __nv_bfloat16*)g, g_ld, gain, (__nv_bfloat16*)out, out_ld, width / parts, eps, scale);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "gated_group_norm: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "gated_group_norm: %s", cudaGetErrorString(e));
    return DL_OK;
}
