// A state-space recurrence with one decay per head and token (the state-space dual form of Mamba-2):
//
//   dt_t = softplus(z_t + dt_bias_h)
//   S_t  = exp(-exp(A_h) dt_t) S_(t-1) + dt_t B_t x_t^T          (S: [state channels, value channels] per head)
//   y_t  = S_t^T C_t + D_h x_t
//
// heads / groups neighbouring heads share a group's B and C.  x, B and C (a short convolution's output, csrc/causal_conv.cu) and
// the step logits z come in the run's type; everything from there on is float32.
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
ssd_scan_kernel(const T* __restrict__ xbc, int ld, const T* __restrict__ z, int z_ld, const float* __restrict__ dt_bias,
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
    const T* x_in = xbc + (size_t)h * P;
    const T* b_in = xbc + (size_t)H * P + (size_t)g * N;
    const T* c_in = b_in + (size_t)G * N;
    T rB[LOADS], rC[LOADS], rx[XLOADS];                        // as loaded: converting here would make the fetch wait for its own loads
    T rz;
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
        rz = z[(size_t)(first + min(tid, count - 1)) * z_ld + h];
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
                sB[buf][e] = live ? dl_to_f32<T>(rB[l]) : 0.f;
                sC[buf][e] = live ? dl_to_f32<T>(rC[l]) : 0.f;
            }
        }
#pragma unroll
        for (int l = 0; l < XLOADS; ++l) sx[buf][tid + SS_THREADS * l] = dl_to_f32<T>(rx[l]);
        if (tid < BATCH) {
            const float dt = ss_softplus(dl_to_f32<T>(rz) + bias);
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
static cudaError_t ssd_launch(const void* xbc, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log,
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
            return dl_launch_dependent_if(early, ssd_scan_kernel<T, ROWS, CPT, true>, grid, block, 0, s, (const T*)xbc, ld, (const T*)z, \
                                          z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, H, \
                                          G, N, P, vec_state);                                                                \
        return dl_launch_dependent_if(early, ssd_scan_kernel<T, ROWS, CPT, false>, grid, block, 0, s, (const T*)xbc, ld, (const T*)z,   \
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

// ---------------------------------------------------------------------------------------------------------------------
// The same recurrence a chunk of SC_L tokens at a time, for prompts of a bfloat16 run: with c_t the running sum of the chunk's
// log decays, S0 the state before the chunk and everything of one head,
//
//   y_t = exp(c_t) S0^T C_t + sum_(j <= t) (C_t . B_j) exp(c_t - c_j) dt_j x_j + D x_t
//   S   = exp(c_L) S0 + sum_j B_j (exp(c_L - c_j) dt_j x_j)^T
//
// so that a chunk is four small matrix products instead of SC_L dependent steps.  B, C and x are bfloat16 (the convolution's
// output in the run's type); decays, steps, sums and the state are float32.  In every product one operand is one of those
// bfloat16 tensors as it is and the other a float32 matrix taken as the sum of three bfloat16 ones (8 + 8 + 8 bits of
// significand), with float32 accumulation: the products are float32 products, run on the tensor cores (mma.sync m16n8k16).
//
// A block owns SC_P value channels of one (sequence, head) and walks the sequence's chunks in order; the state lives in the
// warps' accumulators (warp w holds the row tiles w, w + 4, ..) and goes through shared memory once per chunk as the three
// bfloat16 parts the read-out multiplies with.  Chunks are brought in by cp.async, one ahead; two block barriers a chunk.
#define SC_L 64                          // tokens of a chunk
#define SC_P 32                          // value channels of a block
#define SC_WARPS 4
#define SC_THREADS (32 * SC_WARPS)
#define SC_MAX_STATE 256

__device__ __forceinline__ uint32_t sc_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void sc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sc_ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void sc_ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void sc_copy16(void* dst, const void* src, bool live) {      // 16 bytes, zeros where not live
    const int bytes = live ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(sc_smem(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ float sc_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// v as the sum of three bfloat16 numbers, two values at a time, packed.
__device__ __forceinline__ void sc_split(float v0, float v1, uint32_t (&p)[3]) {
#pragma unroll
    for (int i = 0; i < 3; ++i) {
        const __nv_bfloat162 b = __floats2bfloat162_rn(v0, v1);
        p[i] = *reinterpret_cast<const uint32_t*>(&b);
        v0 -= __low2float(b);
        v1 -= __high2float(b);
    }
}

// Where the walk would leave most of the machine idle (one prompt), the chunks run side by side in three launches instead:
// SC_STATES, every chunk's own contribution to the state, sum_j B_j (exp(c_L - c_j) dt_j x_j)^T, and its whole decay c_L, into
// scratch; ssd_pass_kernel, the states before every chunk one after the other, elementwise, in place; SC_OUTPUTS, every chunk's
// outputs from the state before it.  SC_WALK is the walk in one launch.
enum { SC_WALK = 0, SC_STATES = 1, SC_OUTPUTS = 2 };

template <int NT, int MODE>
__global__ void __launch_bounds__(SC_THREADS)
ssd_chunk_kernel(const __nv_bfloat16* __restrict__ xbc, int ld, const __nv_bfloat16* __restrict__ z, int z_ld, const float* __restrict__ dt_bias,
                 const float* __restrict__ a_log, const float* __restrict__ skip, const int32_t* __restrict__ cu_new,
                 const int32_t* __restrict__ slots, float* __restrict__ state, long slot_stride, int n_slots, float* __restrict__ y, int y_ld,
                 int H, int G, int N, int P, int n_chunks, float* __restrict__ part_state, float* __restrict__ part_decay) {
    constexpr int LDN = NT + 8, LDP = SC_P + 8;               // rows of shared memory, shifted so that ldmatrix misses its own banks
    constexpr int MT = (NT / 16 + SC_WARPS - 1) / SC_WARPS;   // row tiles of the state per warp
    extern __shared__ __align__(128) unsigned char sc_raw[];
    constexpr int BUFS = MODE == SC_WALK ? 2 : 1;             // a walk brings the next chunk while it works on one
    __nv_bfloat16* sB = reinterpret_cast<__nv_bfloat16*>(sc_raw);                 // [BUFS][SC_L][LDN]
    __nv_bfloat16* sC = sB + BUFS * SC_L * LDN;                                   // [BUFS][SC_L][LDN] (not where only states are made)
    __nv_bfloat16* sx = sC + (MODE == SC_STATES ? 0 : BUFS * SC_L * LDN);         // [BUFS][SC_L][LDP]
    __nv_bfloat16* sS = sx + BUFS * SC_L * LDP;                                   // [3][NT][LDP]: the state before the chunk (likewise)
    __nv_bfloat16* sX = sS + (MODE == SC_STATES ? 0 : 3 * NT * LDP);              // [3][SC_L][LDP]: x_j weighted for the new state (not for outputs)
    __shared__ float s_cum[2][SC_L], s_dt[2][SC_L];           // running log2 decay up to and with the token, step size
    dl_launch_dependents();
    const int b = MODE == SC_WALK ? blockIdx.z : blockIdx.z / n_chunks, h = blockIdx.y, g_ = h / (H / G);
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int col0 = blockIdx.x * SC_P;
    const float rate2 = expf(a_log[h]) * 1.4426950408889634f, bias = dt_bias[h], d_skip = skip[h];
    dl_grid_dependency_wait();
    const int t0 = cu_new[b], n = cu_new[b + 1] - t0;
    const int slot = slots[b];
    const int begin = MODE == SC_WALK ? 0 : (blockIdx.z % n_chunks) * SC_L;
    const int end = MODE == SC_WALK ? n : min(n, begin + SC_L);
    if (slot < 0 || slot >= n_slots || begin >= n) return;    // uniform over the block
    const __nv_bfloat16* x_in = xbc + (size_t)t0 * ld + (size_t)h * P + col0;
    const __nv_bfloat16* b_in = xbc + (size_t)t0 * ld + (size_t)H * P + (size_t)g_ * N;
    const __nv_bfloat16* c_in = b_in + (size_t)G * N;
    auto bring = [&](int first, int buf) {                    // the chunk that starts at token `first` of the sequence
        for (int e = tid; e < SC_L * (NT / 8); e += SC_THREADS) {
            const int j = e / (NT / 8), ch = (e - j * (NT / 8)) * 8;
            const bool live = first + j < n && ch < N;
            const size_t at = live ? (size_t)(first + j) * ld + ch : 0;
            sc_copy16(sB + (size_t)(buf * SC_L + j) * LDN + ch, b_in + at, live);
            if (MODE != SC_STATES) sc_copy16(sC + (size_t)(buf * SC_L + j) * LDN + ch, c_in + at, live);
        }
        for (int e = tid; e < SC_L * (SC_P / 8); e += SC_THREADS) {
            const int j = e / (SC_P / 8), ch = (e - j * (SC_P / 8)) * 8;
            const bool live = first + j < n && col0 + ch < P;
            sc_copy16(sx + (size_t)(buf * SC_L + j) * LDP + ch, x_in + (live ? (size_t)(first + j) * ld + ch : 0), live);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    auto scalars = [&](int first, int buf) {                  // warp 0: steps and running log decays; a token that is not there decays nothing
        float dt[2], l[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int j = first + 2 * lane + e;
            dt[e] = j < n ? ss_softplus(__bfloat162float(z[(size_t)(t0 + j) * z_ld + h]) + bias) : 0.f;
            l[e] = -rate2 * dt[e];
        }
        float incl = l[0] + l[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, incl, o);
            if (lane >= o) incl += up;
        }
        float before = __shfl_up_sync(0xffffffffu, incl, 1);
        if (lane == 0) before = 0.f;
        s_cum[buf][2 * lane] = before + l[0];
        s_cum[buf][2 * lane + 1] = before + (l[0] + l[1]);
        s_dt[buf][2 * lane] = dt[0];
        s_dt[buf][2 * lane + 1] = dt[1];
    };
    bring(begin, 0);
    if (warp == 0) scalars(begin, 0);
    // the state: this warp's row tiles, SC_P columns
    float* S = MODE == SC_WALK ? state + (size_t)slot * slot_stride + (size_t)h * N * P : part_state + ((size_t)blockIdx.z * H + h) * N * P;
    float st[MT][SC_P / 8][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = (warp + SC_WARPS * i) * 16 + g + 8 * (e >> 1), col = col0 + c * 8 + 2 * t + (e & 1);
                st[i][c][e] = MODE != SC_STATES && row < N && col < P ? S[(size_t)row * P + col] : 0.f;
            }
    auto put_state = [&]() {                                  // the three parts of this warp's rows into shared memory
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            if (warp + SC_WARPS * i >= NT / 16) continue;
#pragma unroll
            for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
                for (int hf = 0; hf < 2; ++hf) {
                    uint32_t part[3];
                    sc_split(st[i][c][2 * hf], st[i][c][2 * hf + 1], part);
                    const int row = (warp + SC_WARPS * i) * 16 + g + 8 * hf, col = c * 8 + 2 * t;
#pragma unroll
                    for (int q = 0; q < 3; ++q) *reinterpret_cast<uint32_t*>(sS + (size_t)(q * NT + row) * LDP + col) = part[q];
                }
        }
    };
    if (MODE != SC_STATES) put_state();
    // a lane's row and column of the 16 x 16 tile that ldmatrix reads (A as stored; B and the transposed forms share the pattern)
    const int lrow = lane & 15, lcol = (lane >> 4) * 8;
    int buf = 0;
    for (int first = begin; first < end; first += SC_L, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                      // the chunk, its scalars and the state's parts are there; the other buffer is free
        if (first + SC_L < end) bring(first + SC_L, buf ^ 1);
        const __nv_bfloat16* cB = sB + (size_t)buf * SC_L * LDN;
        const __nv_bfloat16* cC = sC + (size_t)buf * SC_L * LDN;
        const __nv_bfloat16* cx = sx + (size_t)buf * SC_L * LDP;
        const float cum_l = s_cum[buf][SC_L - 1];
        // x weighted by what is left of its step at the chunk's end, in three parts
        for (int e = tid; MODE != SC_OUTPUTS && e < SC_L * SC_P / 2; e += SC_THREADS) {
            const int j = e / (SC_P / 2), c = (e - j * (SC_P / 2)) * 2;
            const float w = exp2f(cum_l - s_cum[buf][j]) * s_dt[buf][j];
            const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(cx + (size_t)j * LDP + c);
            uint32_t part[3];
            sc_split(w * __low2float(v), w * __high2float(v), part);
#pragma unroll
            for (int q = 0; q < 3; ++q) *reinterpret_cast<uint32_t*>(sX + (size_t)(q * SC_L + j) * LDP + c) = part[q];
        }
        if (MODE != SC_STATES) {
        // ---- the read-out of the state before the chunk: rows 16 warp .. of C against the state's parts
        float yo[SC_P / 8][4];
#pragma unroll
        for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) yo[c][e] = 0.f;
#pragma unroll 2
        for (int k = 0; k < NT / 16; ++k) {
            uint32_t a[4];
            sc_ldm4(a, sc_smem(cC + (size_t)(16 * warp + lrow) * LDN + 16 * k + lcol));
#pragma unroll
            for (int q = 0; q < 3; ++q)
#pragma unroll
                for (int c2 = 0; c2 < SC_P / 16; ++c2) {
                    uint32_t bb[4];
                    sc_ldm4t(bb, sc_smem(sS + (size_t)(q * NT + 16 * k + lrow) * LDP + 16 * c2 + lcol));
                    sc_mma(yo[2 * c2], a, bb[0], bb[1]);
                    sc_mma(yo[2 * c2 + 1], a, bb[2], bb[3]);
                }
        }
        const int row_lo = 16 * warp + g, row_hi = row_lo + 8;
        const float cum_lo = s_cum[buf][row_lo], cum_hi = s_cum[buf][row_hi];
        const float e_lo = exp2f(cum_lo), e_hi = exp2f(cum_hi);
#pragma unroll
        for (int c = 0; c < SC_P / 8; ++c) yo[c][0] *= e_lo, yo[c][1] *= e_lo, yo[c][2] *= e_hi, yo[c][3] *= e_hi;
        // ---- the chunk's own tokens, sixteen at a time up to the warp's rows
        for (int jb = 0; jb <= warp; ++jb) {
            float gm[2][4];
#pragma unroll
            for (int e = 0; e < 4; ++e) gm[0][e] = gm[1][e] = 0.f;
#pragma unroll 4
            for (int k = 0; k < NT / 16; ++k) {
                uint32_t a[4], bb[4];
                sc_ldm4(a, sc_smem(cC + (size_t)(16 * warp + lrow) * LDN + 16 * k + lcol));
                sc_ldm4(bb, sc_smem(cB + (size_t)(16 * jb + lrow) * LDN + 16 * k + lcol));      // {tokens 0-7, k 0-7}, {8-15, 0-7}, {0-7, 8-15}, {8-15, 8-15}
                sc_mma(gm[0], a, bb[0], bb[2]);
                sc_mma(gm[1], a, bb[1], bb[3]);
            }
            uint32_t parts[3][4];                             // the weights as A operands
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int j = 16 * jb + 8 * hf + 2 * t;
                const float c0 = s_cum[buf][j], c1 = s_cum[buf][j + 1], d0 = s_dt[buf][j], d1 = s_dt[buf][j + 1];
                const float w00 = j <= row_lo ? gm[hf][0] * (sc_ex2(cum_lo - c0) * d0) : 0.f;
                const float w01 = j + 1 <= row_lo ? gm[hf][1] * (sc_ex2(cum_lo - c1) * d1) : 0.f;
                const float w10 = j <= row_hi ? gm[hf][2] * (sc_ex2(cum_hi - c0) * d0) : 0.f;
                const float w11 = j + 1 <= row_hi ? gm[hf][3] * (sc_ex2(cum_hi - c1) * d1) : 0.f;
                uint32_t lo[3], hi[3];
                sc_split(w00, w01, lo);
                sc_split(w10, w11, hi);
#pragma unroll
                for (int q = 0; q < 3; ++q) parts[q][2 * hf] = lo[q], parts[q][2 * hf + 1] = hi[q];
            }
#pragma unroll
            for (int c2 = 0; c2 < SC_P / 16; ++c2) {
                uint32_t bb[4];
                sc_ldm4t(bb, sc_smem(cx + (size_t)(16 * jb + lrow) * LDP + 16 * c2 + lcol));
#pragma unroll
                for (int q = 0; q < 3; ++q) {
                    sc_mma(yo[2 * c2], parts[q], bb[0], bb[1]);
                    sc_mma(yo[2 * c2 + 1], parts[q], bb[2], bb[3]);
                }
            }
        }
#pragma unroll
        for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {
                const int j = hf ? row_hi : row_lo, col = c * 8 + 2 * t;
                if (first + j < n && col0 + col < P) {         // P is even: pairs are whole
                    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(cx + (size_t)j * LDP + col);
                    *reinterpret_cast<float2*>(y + (size_t)(t0 + first + j) * y_ld + (size_t)h * P + col0 + col) =
                        make_float2(fmaf(d_skip, __low2float(v), yo[c][2 * hf]), fmaf(d_skip, __high2float(v), yo[c][2 * hf + 1]));
                }
            }
        }
        if (MODE == SC_OUTPUTS) return;
        __syncthreads();                                      // the weighted x is there; everyone is done with the state's parts
        // ---- the new state
        const float keep = exp2f(cum_l);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            if (warp + SC_WARPS * i >= NT / 16) continue;
#pragma unroll
            for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
                for (int e = 0; e < 4; ++e) st[i][c][e] *= keep;
#pragma unroll
            for (int k = 0; k < SC_L / 16; ++k) {
                uint32_t a[4], at[4];
                sc_ldm4t(at, sc_smem(cB + (size_t)(16 * k + lrow) * LDN + 16 * (warp + SC_WARPS * i) + lcol));
                a[0] = at[0], a[1] = at[2], a[2] = at[1], a[3] = at[3];   // read as {k 0-7, m 0-7}, {k 8-15, m 0-7}, {k 0-7, m 8-15}, {k 8-15, m 8-15}
#pragma unroll
                for (int q = 0; q < 3; ++q)
#pragma unroll
                    for (int c2 = 0; c2 < SC_P / 16; ++c2) {
                        uint32_t bb[4];
                        sc_ldm4t(bb, sc_smem(sX + (size_t)(q * SC_L + 16 * k + lrow) * LDP + 16 * c2 + lcol));
                        sc_mma(st[i][2 * c2], a, bb[0], bb[1]);
                        sc_mma(st[i][2 * c2 + 1], a, bb[2], bb[3]);
                    }
            }
        }
        if (first + SC_L < end) {
            put_state();
            if (warp == 0) scalars(first + SC_L, buf ^ 1);
        }
    }
    if (MODE == SC_STATES && tid == 0 && blockIdx.x == 0) part_decay[(size_t)blockIdx.z * H + h] = s_cum[0][SC_L - 1];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int c = 0; c < SC_P / 8; ++c)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int row = (warp + SC_WARPS * i) * 16 + g + 8 * (e >> 1), col = col0 + c * 8 + 2 * t + (e & 1);
                if (row < N && col < P) S[(size_t)row * P + col] = st[i][c][e];
            }
}

// The state before every chunk, in place of the chunk's contribution: four neighbouring values of one (sequence, head) a thread.
__global__ void __launch_bounds__(256)
ssd_pass_kernel(float* __restrict__ part_state, const float* __restrict__ part_decay, const int32_t* __restrict__ cu_new,
                const int32_t* __restrict__ slots, float* __restrict__ state, long slot_stride, int n_slots, int H, int NP, int n_chunks) {
    dl_launch_dependents();
    dl_grid_dependency_wait();
    const int b = blockIdx.z, h = blockIdx.y, at = (blockIdx.x * 256 + threadIdx.x) * 4;
    const int n = cu_new[b + 1] - cu_new[b], slot = slots[b];
    if (at >= NP || n <= 0 || slot < 0 || slot >= n_slots) return;
    const int chunks = (n + SC_L - 1) / SC_L;
    float4* S = reinterpret_cast<float4*>(state + (size_t)slot * slot_stride + (size_t)h * NP + at);
    float4 s = *S;
    float* p = part_state + ((size_t)b * n_chunks * H + h) * NP + at;
    const float* d = part_decay + (size_t)b * n_chunks * H + h;
    const size_t step = (size_t)H * NP;
    constexpr int AHEAD = 8;                                 // chunks whose contributions are asked for together
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float4 v[AHEAD];
        float k[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const int c = min(c0 + i, chunks - 1);
            v[i] = *reinterpret_cast<const float4*>(p + (size_t)c * step);
            k[i] = d[(size_t)c * H];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            if (c0 + i >= chunks) break;
            *reinterpret_cast<float4*>(p + (size_t)(c0 + i) * step) = s;
            const float keep = exp2f(k[i]);
            s = make_float4(fmaf(keep, s.x, v[i].x), fmaf(keep, s.y, v[i].y), fmaf(keep, s.z, v[i].z), fmaf(keep, s.w, v[i].w));
        }
    }
    *S = s;
}

template <int NT, int MODE>
static cudaError_t ssd_chunk_go(dim3 grid, const void* xbc, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log,
                                const float* skip, const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride, int n_slots,
                                float* y, int y_ld, int H, int G, int N, int P, int n_chunks, float* part_state, float* part_decay,
                                cudaStream_t s) {
    constexpr int bufs = MODE == SC_WALK ? 2 : 1;
    const size_t smem = (size_t)(bufs * SC_L * ((MODE == SC_STATES ? 1 : 2) * (NT + 8) + SC_P + 8) + (MODE == SC_STATES ? 0 : 3 * NT * (SC_P + 8)) +
                                 (MODE == SC_OUTPUTS ? 0 : 3 * SC_L * (SC_P + 8))) * 2;
    static bool configured = false;
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(ssd_chunk_kernel<NT, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
        configured = true;
    }
    const bool early = (long)grid.x * grid.y * grid.z > 2L * dl_sm_count();
    return dl_launch_dependent_if(early, ssd_chunk_kernel<NT, MODE>, grid, dim3(SC_THREADS), smem, s, (const __nv_bfloat16*)xbc, ld,
                                  (const __nv_bfloat16*)z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, H, G, N, P,
                                  n_chunks, part_state, part_decay);
}

template <int NT>
static int ssd_chunk_launch(const void* xbc, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log, const float* skip,
                            const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride, int n_slots, float* y, int y_ld,
                            int n_seqs, int H, int G, int N, int P, int n_chunks, float* part_state, float* part_decay, cudaStream_t s) {
    const dim3 walk((P + SC_P - 1) / SC_P, H, n_seqs), side(walk.x, H, n_seqs * n_chunks);
    cudaError_t e;
#define SC_ARGS xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, H, G, N, P, n_chunks, part_state, part_decay, s
    if (part_state == nullptr) {
        e = ssd_chunk_go<NT, SC_WALK>(walk, SC_ARGS);
    } else {
        e = ssd_chunk_go<NT, SC_STATES>(side, SC_ARGS);
        if (e == cudaSuccess)
            e = dl_launch_dependent(ssd_pass_kernel, dim3((N * P / 4 + 255) / 256, H, n_seqs), dim3(256), 0, s, part_state, (const float*)part_decay,
                                    cu_new, slots, state, slot_stride, n_slots, H, N * P, n_chunks);
        if (e == cudaSuccess) e = ssd_chunk_go<NT, SC_OUTPUTS>(side, SC_ARGS);
    }
#undef SC_ARGS
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "ssd_chunk: %s", cudaGetErrorString(e));
    return DL_OK;
}

// As dl_ssd_scan, a chunk at a time on the tensor cores: xbc and z bfloat16, rows and their parts 16-byte aligned (ld, N and P
// multiples of 8), N up to SC_MAX_STATE.  part_state float32 [n_seqs * n_chunks, H, N, P] and part_decay float32 [n_seqs * n_chunks, H]
// (n_chunks: SC_L-token chunks of the longest sequence): the chunks run side by side; both NULL: a block walks its sequence's chunks.
extern "C" int dl_ssd_chunk(const void* xbc, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log, const float* skip,
                            const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride, int n_slots, float* y, int y_ld,
                            int n_seqs, int H, int G, int N, int P, int n_chunks, float* part_state, float* part_decay, void* stream) {
    DL_REQUIRE(n_seqs >= 0 && H > 0 && G > 0 && N > 0 && P > 0 && n_slots > 0 && H % G == 0 && H <= 65535 && n_seqs <= 65535, "ssd_chunk: bad sizes");
    DL_REQUIRE((part_state == nullptr) == (part_decay == nullptr) &&
                   (part_state == nullptr || (n_chunks >= 1 && (long)n_seqs * n_chunks <= 65535 && slot_stride % 4 == 0 && ((uintptr_t)state % 16) == 0 &&
                                              ((uintptr_t)part_state % 16) == 0)),
               "ssd_chunk: chunks side by side need scratch for at most 65,535 of them and aligned states");
    DL_REQUIRE(N % 8 == 0 && P % 8 == 0 && ld % 8 == 0 && ((uintptr_t)xbc % 16) == 0 && N <= SC_MAX_STATE && y_ld % 2 == 0 && ((uintptr_t)y % 8) == 0,
               "ssd_chunk: state and value channels come in aligned eights, the state up to %d", SC_MAX_STATE);
    DL_REQUIRE(ld >= H * P + 2 * G * N && z_ld >= H && y_ld >= H * P && slot_stride >= (long)H * N * P, "ssd_chunk: rows overlap");
    if (n_seqs == 0) return DL_OK;
#define SC_GO(NT) return ssd_chunk_launch<NT>(xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, n_seqs, H, G, N, P, n_chunks, part_state, part_decay, (cudaStream_t)stream)
    if (N <= 32) SC_GO(32);
    if (N <= 64) SC_GO(64);
    if (N <= 128) SC_GO(128);
    SC_GO(256);
#undef SC_GO
}

// xbc [tokens, H*P + 2*G*N] of dtype (rows ld apart): x, then B, then C; z [tokens, H] of dtype (rows z_ld apart): the step logits; dt_bias, a_log, skip float32 [H]; state float32 [N, P] per head at `state` + slot * slot_stride; y float32 [tokens, H*P].
extern "C" int dl_ssd_scan(const void* xbc, int dtype, int ld, const void* z, int z_ld, const float* dt_bias, const float* a_log,
                           const float* skip, const int32_t* cu_new, const int32_t* slots, float* state, long slot_stride,
                           int n_slots, float* y, int y_ld, int n_seqs, int n_tokens, int H, int G, int N, int P, void* stream) {
    DL_REQUIRE(n_seqs >= 0 && n_tokens >= 0 && H > 0 && G > 0 && N > 0 && P > 0 && n_slots > 0 && H % G == 0, "ssd_scan: bad sizes");
    DL_REQUIRE(N <= SS_MAX_STATE, "ssd_scan: a state of %d channels, the kernel takes up to %d", N, SS_MAX_STATE);
    DL_REQUIRE(ld >= H * P + 2 * G * N && z_ld >= H && y_ld >= H * P && slot_stride >= (long)H * N * P, "ssd_scan: rows overlap");
    DL_REQUIRE(H <= 65535 && n_seqs <= 65535, "ssd_scan: too many heads or sequences");
    if (n_seqs == 0 || n_tokens == 0) return DL_OK;
    cudaError_t e;
    if (dtype == DL_F32)
        e = ssd_launch<float>(xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, n_seqs, n_tokens, H, G, N, P, (cudaStream_t)stream);
    else if (dtype == DL_BF16)
        e = ssd_launch<__nv_bfloat16>(xbc, ld, z, z_ld, dt_bias, a_log, skip, cu_new, slots, state, slot_stride, n_slots, y, y_ld, n_seqs, n_tokens, H, G, N, P, (cudaStream_t)stream);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "ssd_scan: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "ssd_scan: %s", cudaGetErrorString(e));
    return DL_OK;
}

// A gate in front of a norm over equal parts of a row:
//   v = y * silu(g);  out = scale * v / sqrt(mean over the part of v^2 + eps) * gain
// One block per (row, part).  y float32, g of the step's type, float32 arithmetic; rows of g and out may be column views.
#define GN_THREADS 256
#define GN_BIG 1024

__device__ __forceinline__ float gn_silu(float v) { return v / (1.0f + expf(-v)); }
__device__ __forceinline__ float4 gn_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 gn_load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}
__device__ __forceinline__ void gn_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void gn_store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&a);
    raw.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// NV pieces of four per thread in registers.
template <typename T, int THREADS, int NV>
__global__ void __launch_bounds__(THREADS)
gated_group_norm_vec_kernel(const float* __restrict__ y, int y_ld, const T* __restrict__ g, int g_ld, const float* __restrict__ gain,
                            T* __restrict__ out, int out_ld, int part, float eps, float scale) {
    __shared__ float scratch[33];
    dl_launch_dependents();
    const int c0 = blockIdx.y * part;
    float4 w[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {                           // weights: no kernel of the stream writes them
        const int c = (threadIdx.x + i * THREADS) * 4;
        w[i] = c < part ? gn_load4(gain + c0 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    dl_grid_dependency_wait();
    const float* yr = y + (size_t)blockIdx.x * y_ld + c0;
    const T* gr = g + (size_t)blockIdx.x * g_ld + c0;
    T* dst = out + (size_t)blockIdx.x * out_ld + c0;
    float4 v[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < part) {
            const float4 a = gn_load4(yr + c), b = gn_load4(gr + c);
            v[i] = make_float4(a.x * gn_silu(b.x), a.y * gn_silu(b.y), a.z * gn_silu(b.z), a.w * gn_silu(b.w));
        }
        ss += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
    }
    ss = dl_block_sum(ss, scratch);
    const float r = scale / sqrtf(ss / (float)part + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (threadIdx.x + i * THREADS) * 4;
        if (c < part) gn_store4(dst + c, make_float4(v[i].x * r * w[i].x, v[i].y * r * w[i].y, v[i].z * r * w[i].z, v[i].w * r * w[i].w));
    }
}

// Any part: every value is computed twice.
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
    float ss = 0.f;
    for (int c = threadIdx.x; c < part; c += GN_THREADS) { const float w = yr[c] * gn_silu(dl_to_f32<T>(gr[c])); ss += w * w; }
    ss = dl_block_sum(ss, scratch);
    const float r = scale / sqrtf(ss / (float)part + eps);
    for (int c = threadIdx.x; c < part; c += GN_THREADS) dst[c] = dl_from_f32<T>(yr[c] * gn_silu(dl_to_f32<T>(gr[c])) * r * gain[c0 + c]);
}

template <typename T>
static cudaError_t gn_launch(const float* y, int y_ld, const void* g, int g_ld, const float* gain, void* out, int out_ld, int rows, int width,
                             int parts, float eps, float scale, cudaStream_t s) {
    const int part = width / parts;
    const size_t quad = 4 * sizeof(T);
    const bool vec = part % 4 == 0 && y_ld % 4 == 0 && g_ld % 4 == 0 && out_ld % 4 == 0 && ((uintptr_t)y % 16) == 0 && ((uintptr_t)gain % 16) == 0 &&
                     ((uintptr_t)g % quad) == 0 && ((uintptr_t)out % quad) == 0 && part <= GN_BIG * 4 * 4;
    const dim3 grid(rows, parts);
#define GN_GO(TH, NV) return dl_launch_dependent(gated_group_norm_vec_kernel<T, TH, NV>, grid, dim3(TH), 0, s, y, y_ld, (const T*)g, g_ld, gain, (T*)out, out_ld, part, eps, scale)
    if (vec && part <= GN_THREADS * 4) GN_GO(GN_THREADS, 1);
    const bool few = (long)rows * parts <= 2 * dl_sm_count();
    if (vec && !few && part <= GN_THREADS * 8) GN_GO(GN_THREADS, 2);
    if (vec && !few && part <= GN_THREADS * 16) GN_GO(GN_THREADS, 4);
    if (vec && part <= GN_BIG * 4) GN_GO(GN_BIG, 1);
    if (vec) GN_GO(GN_BIG, 4);
#undef GN_GO
    return dl_launch_dependent(gated_group_norm_kernel<T>, grid, dim3(GN_THREADS), 0, s, y, y_ld, (const T*)g, g_ld, gain, (T*)out, out_ld, part, eps, scale);
}

extern "C" int dl_gated_group_norm(const float* y, int y_ld, const void* g, int g_ld, const float* gain, void* out, int out_ld,
                                   int dtype, int rows, int width, int parts, float eps, float scale, void* stream) {
    DL_REQUIRE(rows >= 0 && width > 0 && parts > 0 && width % parts == 0 && parts <= 65535 && eps > 0.f, "gated_group_norm: bad sizes");
    DL_REQUIRE(y_ld >= width && g_ld >= width && out_ld >= width, "gated_group_norm: rows overlap");
    if (rows == 0) return DL_OK;
    cudaError_t e;
    if (dtype == DL_F32) e = gn_launch<float>(y, y_ld, g, g_ld, gain, out, out_ld, rows, width, parts, eps, scale, (cudaStream_t)stream);
    else if (dtype == DL_BF16) e = gn_launch<__nv_bfloat16>(y, y_ld, g, g_ld, gain, out, out_ld, rows, width, parts, eps, scale, (cudaStream_t)stream);
    else
        return dl_fail(DL_ERR_UNSUPPORTED, "gated_group_norm: dtype %d", dtype);
    if (e != cudaSuccess) return dl_fail(DL_ERR_LAUNCH, "gated_group_norm: %s", cudaGetErrorString(e));
    return DL_OK;
}
