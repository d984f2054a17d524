// The residual of a pre-norm decoder kept as ONE float32 stream, with everything that may lie between two sublayers in one
// kernel. With y the output of the sublayer before (compute dtype or float32):
//     x <- x + factor * (scale * y)          scale: a number per feature ("layer scale"), factor: a constant
//     x <- x + factor * y2                   y2: the output of a second sublayer that read the same input, either rows like y or
//                                            a mixture's experts: moe_weight * sum_c moe_rows[moe_slots[t][c]] (float32 rows in
//                                            expert order, the weighted sum with equal weights, made here and never stored)
//     x <- x + add_rows[t] + add_vec         what a pass over a stretch of layers starts with (both optional)
//     h  = norm_w * x / sqrt(mean(x^2) + eps)
// and, with a token shift, h_t <- h_t + (h_(t-1) - h_t) * shift per feature, where h_(t-1) is the request's token before as
// it was BEFORE this replacement (zeros for its first token). The h of a request's last token of a step is kept, float32 and
// unrounded, in the request's state slot, so a token's result is the same bits whatever the cut.
//
// The token before may lie in another block, and its row of x is being updated in the same launch. So the shifted form reads
// x_in and writes x_out, two buffers, and a block works the row before its own out again (it is read from L2 and normed a
// second time, never stored twice). A block takes R neighbouring tokens, so one row in R is worked out twice. The slot of a
// request is read by its first token of the step and takes the h of its last: the block of the FIRST token does both, in
// that order and feature by feature in the same thread, so no block has to wait for another.
// Sums, norm and shift are float32; the rounding of h to the compute dtype is the only one.
#include "common.cuh"

struct StreamStepArgs {
    const float* x_in;
    float* x_out;                          // may be x_in without a shift; null: the updated rows are not kept
    const void* y; const float* y_scale; float y_factor;
    const void* y2;
    const float* moe_rows; const int* moe_slots; int moe_top; float moe_weight;
    const float *add_rows, *add_vec;
    const float* norm_w; float eps;
    void* h;
    const int* rows;                       // without a shift: the tokens to work on (h has a row per entry), or null
    const float* shift; float* prev; long long prev_stride;      // prev: slot s at prev + s * prev_stride, [width]
    const int *token_seq, *cu_seqlens, *state_slots;
    int num_tokens, width;
};

template <int VEC> struct SsVec;
template <> struct SsVec<1> {
    static __device__ __forceinline__ void load(const float* p, float* v) { v[0] = *p; }
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) { v[0] = __bfloat162float(*p); }
    static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct SsVec<4> {
    static __device__ __forceinline__ void load(const float* p, float* v) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
    }
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* v) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
        v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
    }
    static __device__ __forceinline__ void store(float* p, const float* v) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) {
        uint2 u;
        *reinterpret_cast<__nv_bfloat162*>(&u.x) = __floats2bfloat162_rn(v[0], v[1]);
        *reinterpret_cast<__nv_bfloat162*>(&u.y) = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2*>(p) = u;
    }
};

// Features i .. i + VEC of the updated row t.
template <typename TY, int VEC>
__device__ __forceinline__ void updated_row(const StreamStepArgs& a, size_t t, int i, float* u) {
    SsVec<VEC>::load(a.x_in + t * a.width + i, u);
    if (a.y) {
        float y[VEC], s[VEC];
        SsVec<VEC>::load((const TY*)a.y + t * a.width + i, y);
        if (a.y_scale) {
            SsVec<VEC>::load(a.y_scale + i, s);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] *= s[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = fmaf(a.y_factor, y[e], u[e]);
    }
    if (a.y2) {
        float y[VEC];
        SsVec<VEC>::load((const TY*)a.y2 + t * a.width + i, y);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = fmaf(a.y_factor, y[e], u[e]);
    }
    if (a.moe_rows) {
        float y[VEC] = {};
        for (int c = 0; c < a.moe_top; ++c) {
            float r[VEC];
            SsVec<VEC>::load(a.moe_rows + (size_t)a.moe_slots[t * a.moe_top + c] * a.width + i, r);
#pragma unroll
            for (int e = 0; e < VEC; ++e) y[e] += r[e];
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = fmaf(a.y_factor * a.moe_weight, y[e], u[e]);
    }
    if (a.add_rows) {
        float r[VEC];
        SsVec<VEC>::load(a.add_rows + t * a.width + i, r);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] += r[e];
    }
    if (a.add_vec) {
        float r[VEC];
        SsVec<VEC>::load(a.add_vec + i, r);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] += r[e];
    }
}

constexpr int SS_MAX_THREADS = 256;

template <typename TY, typename TH, int VEC>
__global__ void __launch_bounds__(SS_MAX_THREADS) stream_step_kernel(StreamStepArgs a) {
    extern __shared__ __align__(16) float ss_buf[];
    __shared__ float red[33];
    ti_grid_launch_dependents();
    ti_grid_wait();
    const int r = blockIdx.x;
    const size_t t = a.rows ? a.rows[r] : r;
    float ss = 0.f;
    for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
        float u[VEC];
        updated_row<TY, VEC>(a, t, i, u);
        if (a.x_out) SsVec<VEC>::store(a.x_out + t * a.width + i, u);
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(u[e], u[e], ss);
        SsVec<VEC>::store(ss_buf + i, u);
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)a.width + a.eps);
    for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
        float u[VEC], w[VEC];
        SsVec<VEC>::load(ss_buf + i, u);
        SsVec<VEC>::load(a.norm_w + i, w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u[e] = w[e] * u[e] * inv;
        SsVec<VEC>::store((TH*)a.h + (size_t)r * a.width + i, u);
    }
}

// Rows of the buffer: 0 the token before the block's first (if it belongs to the same request), 1 .. R the block's own.
template <typename TY, typename TH, int VEC, int R>
__global__ void __launch_bounds__(SS_MAX_THREADS) stream_shift_kernel(StreamStepArgs a) {
    extern __shared__ __align__(16) float ss_buf[];                // [R + 1][width]; a thread only touches its own features
    __shared__ float red[R + 1][SS_MAX_THREADS / 32];
    __shared__ float red1[33];
    ti_grid_launch_dependents();
    ti_grid_wait();
    const int t0 = blockIdx.x * R, n = min(R, a.num_tokens - t0);
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    bool first[R];                                                 // the token is its request's first of the step
    int seqs[R];
#pragma unroll
    for (int j = 0; j < R; ++j) {
        seqs[j] = j < n ? a.token_seq[t0 + j] : 0;
        first[j] = j < n && a.cu_seqlens[seqs[j]] == t0 + j;
    }
    const bool halo = !first[0];
    float ss[R + 1];
#pragma unroll
    for (int j = 0; j <= R; ++j) ss[j] = 0.f;
    for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
#pragma unroll
        for (int j = 0; j <= R; ++j) {
            if (j == 0 ? !halo : j > n) continue;
            const size_t t = (size_t)(t0 + j) - 1;
            float u[VEC];
            updated_row<TY, VEC>(a, t, i, u);
            if (a.x_out && j > 0) SsVec<VEC>::store(a.x_out + t * a.width + i, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss[j] = fmaf(u[e], u[e], ss[j]);
            SsVec<VEC>::store(ss_buf + (size_t)j * a.width + i, u);
        }
    }
#pragma unroll
    for (int j = 0; j <= R; ++j) {
        const float v = warp_sum(ss[j]);
        if (lane == 0) red[j][warp] = v;
    }
    __syncthreads();
    float inv[R + 1];
#pragma unroll
    for (int j = 0; j <= R; ++j) {
        float v = 0.f;
        for (int w = 0; w < warps; ++w) v += red[j][w];
        inv[j] = rsqrtf(v / (float)a.width + a.eps);
    }
    for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
        float w[VEC], sh[VEC], before[VEC];
        SsVec<VEC>::load(a.norm_w + i, w);
        SsVec<VEC>::load(a.shift + i, sh);
        if (halo) {
            SsVec<VEC>::load(ss_buf + i, before);
#pragma unroll
            for (int e = 0; e < VEC; ++e) before[e] = w[e] * before[e] * inv[0];
        }
#pragma unroll
        for (int j = 0; j < R; ++j) {
            if (j >= n) continue;
            float h[VEC], o[VEC];
            SsVec<VEC>::load(ss_buf + (size_t)(j + 1) * a.width + i, h);
#pragma unroll
            for (int e = 0; e < VEC; ++e) h[e] = w[e] * h[e] * inv[j + 1];
            if (first[j]) {
                float* slot = a.prev + (size_t)a.state_slots[seqs[j]] * a.prev_stride + i;
                SsVec<VEC>::load(slot, before);
                if (a.cu_seqlens[seqs[j] + 1] == t0 + j + 1) SsVec<VEC>::store(slot, h);      // the request's only token
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                o[e] = fmaf(before[e] - h[e], sh[e], h[e]);
                before[e] = h[e];
            }
            SsVec<VEC>::store((TH*)a.h + (size_t)(t0 + j) * a.width + i, o);
        }
    }
    // requests that start in this block and bring more than one token: their slot takes the h of their last one
#pragma unroll 1
    for (int j = 0; j < n; ++j) {
        const int seq = a.token_seq[t0 + j];
        const int last = a.cu_seqlens[seq + 1] - 1;
        if (a.cu_seqlens[seq] != t0 + j || last == t0 + j) continue;
        float sl = 0.f;
        for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
            float u[VEC];
            updated_row<TY, VEC>(a, last, i, u);
#pragma unroll
            for (int e = 0; e < VEC; ++e) sl = fmaf(u[e], u[e], sl);
            SsVec<VEC>::store(ss_buf + i, u);
        }
        // the sum in the order of the rows above: warp by warp
        const float v = warp_sum(sl);
        __syncthreads();
        if (lane == 0) red1[warp] = v;
        __syncthreads();
        float tot = 0.f;
        for (int w = 0; w < warps; ++w) tot += red1[w];
        const float il = rsqrtf(tot / (float)a.width + a.eps);
        float* slot = a.prev + (size_t)a.state_slots[seq] * a.prev_stride;
        for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
            float u[VEC], w[VEC];
            SsVec<VEC>::load(ss_buf + i, u);
            SsVec<VEC>::load(a.norm_w + i, w);
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] = w[e] * u[e] * il;
            SsVec<VEC>::store(slot + i, u);
        }
    }
}

// What a pass over a stretch of layers projects: the updated row beside the embedding's, as the operand row of a product. In
// bfloat16 the float32 row travels as two halves, u = hi + lo (16 bits of mantissa instead of 8; the product's weight has the
// columns for it twice): out row [hi | lo | x0]. In float32: [u | x0]. x0 = scale * table[token].
template <typename TY, typename TO, int VEC>
__global__ void __launch_bounds__(SS_MAX_THREADS) stream_enter_kernel(StreamStepArgs a, TO* __restrict__ out, const TO* __restrict__ table,
                                                                      const int* __restrict__ token_ids, int vocab, float scale) {
    ti_grid_launch_dependents();
    ti_grid_wait();
    const size_t t = blockIdx.x;
    const int token = token_ids[t];
    const bool known = token >= 0 && token < vocab;
    constexpr int PARTS = sizeof(TO) == 4 ? 2 : 3;
    TO* row = out + t * PARTS * a.width;
    for (int i = threadIdx.x * VEC; i < a.width; i += blockDim.x * VEC) {
        float u[VEC], x0[VEC] = {};
        updated_row<TY, VEC>(a, t, i, u);
        if (known) SsVec<VEC>::load(table + (size_t)token * a.width + i, x0);
#pragma unroll
        for (int e = 0; e < VEC; ++e) x0[e] *= scale;
        SsVec<VEC>::store(row + i, u);
        if constexpr (PARTS == 3) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] -= to_f32(from_f32<TO>(u[e]));
            SsVec<VEC>::store(row + a.width + i, u);
        }
        SsVec<VEC>::store(row + (PARTS - 1) * a.width + i, x0);
    }
}

template <typename K>
static int ss_smem(K kernel, size_t bytes) {
    if (bytes <= 40 * 1024) return 0;             // with the static arrays still under what needs no opt-in
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    TI_REQUIRE(e == cudaSuccess, "stream_step: cannot get %d bytes of shared memory: %s", (int)bytes, cudaGetErrorString(e));
    return 0;
}

// out [num_tokens][3 width] (bfloat16) or [num_tokens][2 width] (float32, dtype); the updates as in ti_stream_step.
TI_API int ti_stream_enter(void* out, const float* x_in, const void* y, const float* y_scale, float y_factor, const void* y2,
                           const float* moe_rows, const int* moe_slots, int moe_top, float moe_weight, const float* add_rows,
                           const float* add_vec, const void* table, const int* token_ids, int vocab, float scale, int num_tokens,
                           int width, int y_dtype, int dtype, cudaStream_t stream) {
    TI_REQUIRE(num_tokens >= 0 && width > 0 && vocab > 0 && out && x_in && table && token_ids, "stream_enter: bad arguments");
    TI_REQUIRE(!moe_rows || (moe_slots && moe_top > 0), "stream_enter: experts' rows come with their slots");
    if (num_tokens == 0) return 0;
    StreamStepArgs a = {x_in, nullptr, y, y_scale, y_factor, y2, moe_rows, moe_slots, moe_top, moe_weight, add_rows, add_vec, nullptr,
                        0.f, nullptr, nullptr, nullptr, nullptr, 0, nullptr, nullptr, nullptr, num_tokens, width};
    const uintptr_t all = (uintptr_t)x_in | (uintptr_t)y | (uintptr_t)y_scale | (uintptr_t)y2 | (uintptr_t)moe_rows |
                          (uintptr_t)add_rows | (uintptr_t)add_vec | (uintptr_t)table | (uintptr_t)out;
    const bool wide = width % 4 == 0 && all % 16 == 0;
    int threads = 64;
    while (threads < SS_MAX_THREADS && threads * 4 < width) threads <<= 1;
    typedef __nv_bfloat16 B;
#define SE_GO(TY, TO)                                                                                                             \
    do {                                                                                                                          \
        if (wide) ti_launch(stream_enter_kernel<TY, TO, 4>, num_tokens, threads, 0, stream, a, (TO*)out, (const TO*)table, token_ids, vocab, scale); \
        else ti_launch(stream_enter_kernel<TY, TO, 1>, num_tokens, threads, 0, stream, a, (TO*)out, (const TO*)table, token_ids, vocab, scale);      \
    } while (0)
    if (y_dtype == TI_F32 && dtype == TI_F32) SE_GO(float, float);
    else if (y_dtype == TI_F32 && dtype == TI_BF16) SE_GO(float, B);
    else if (y_dtype == TI_BF16 && dtype == TI_BF16) SE_GO(B, B);
    else TI_REQUIRE(false, "stream_enter: unknown dtypes %d, %d", y_dtype, dtype);
#undef SE_GO
    TI_CHECK_LAUNCH("stream_enter");
    return 0;
}

// x_in, x_out float32 [num_tokens][width] (x_out null: not kept; with a shift it is not x_in). y (or null) with y_scale
// (float32 [width], or null) and y_factor; y2 (of y's dtype, or null), moe_rows float32 [slots][width] with moe_slots
// [num_tokens][moe_top] and moe_weight (or null); add_rows float32 [num_tokens][width], add_vec float32 [width] (or null). h:
// [num_rows][width]. shift (float32 [width], or null) with prev (slots of `width` floats, prev_stride apart), token_seq,
// cu_seqlens and state_slots of the step.
TI_API int ti_stream_step(const float* x_in, float* x_out, const void* y, const float* y_scale, float y_factor, const void* y2,
                          const float* moe_rows, const int* moe_slots, int moe_top, float moe_weight, const float* add_rows, const float* add_vec, const float* norm_w, float eps, void* h, const int* rows,
                          int num_rows, const float* shift, float* prev, long long prev_stride, const int* token_seq,
                          const int* cu_seqlens, const int* state_slots, int num_tokens, int width, int y_dtype, int h_dtype,
                          cudaStream_t stream) {
    TI_REQUIRE(num_rows >= 0 && num_tokens >= 0 && width > 0 && width <= 24 * 1024, "stream_step: bad sizes");
    TI_REQUIRE(x_in && norm_w && h, "stream_step: the stream, the norm and the output are needed");
    TI_REQUIRE(!shift || (!rows && num_rows == num_tokens && prev && token_seq && cu_seqlens && state_slots && x_out != x_in),
               "stream_step: a token shift works on all of a step's tokens, from one buffer into another");
    TI_REQUIRE(!rows || !x_out, "stream_step: chosen rows are not stored back");
    TI_REQUIRE(!moe_rows || (moe_slots && moe_top > 0), "stream_step: experts' rows come with their slots");
    if (num_rows == 0) return 0;
    StreamStepArgs a = {x_in, x_out, y, y_scale, y_factor, y2, moe_rows, moe_slots, moe_top, moe_weight, add_rows, add_vec, norm_w, eps, h, rows, shift, prev, prev_stride,
                        token_seq, cu_seqlens, state_slots, num_tokens, width};
    const uintptr_t all = (uintptr_t)x_in | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)y_scale | (uintptr_t)y2 | (uintptr_t)moe_rows |
                          (uintptr_t)add_rows | (uintptr_t)add_vec | (uintptr_t)norm_w | (uintptr_t)h | (uintptr_t)shift | (uintptr_t)prev;
    const bool wide = width % 4 == 0 && all % 16 == 0 && (!shift || prev_stride % 4 == 0);
    int threads = 64;
    while (threads < SS_MAX_THREADS && threads * 4 < width) threads <<= 1;
    typedef __nv_bfloat16 B;
    // three tokens a block (a row in three worked out twice) where that still leaves every SM blocks enough
    const int per_block = shift && num_tokens >= 3 * 148 * 2 && (size_t)width * 16 <= 48 * 1024 ? 3 : 1;
    const size_t smem = (size_t)width * sizeof(float) * (shift ? per_block + 1 : 1);
#define SS_GO(K, blocks)                                        \
    do {                                                        \
        if (ss_smem(K, smem)) return -1;                        \
        ti_launch(K, (blocks), threads, smem, stream, a);       \
    } while (0)
#define SS_V(TY, TH, VEC)                                                                                                  \
    do {                                                                                                                   \
        if (!shift) SS_GO((stream_step_kernel<TY, TH, VEC>), num_rows);                                                    \
        else if (per_block == 3) SS_GO((stream_shift_kernel<TY, TH, VEC, 3>), (num_tokens + 2) / 3);                       \
        else SS_GO((stream_shift_kernel<TY, TH, VEC, 1>), num_tokens);                                                     \
    } while (0)
#define SS_T(TY, TH)                  \
    do {                              \
        if (wide) SS_V(TY, TH, 4);    \
        else SS_V(TY, TH, 1);         \
    } while (0)
    if (y_dtype == TI_F32 && h_dtype == TI_F32) SS_T(float, float);
    else if (y_dtype == TI_F32 && h_dtype == TI_BF16) SS_T(float, B);
    else if (y_dtype == TI_BF16 && h_dtype == TI_BF16) SS_T(B, B);
    else TI_REQUIRE(false, "stream_step: unknown dtypes %d, %d", y_dtype, h_dtype);
#undef SS_T
#undef SS_V
#undef SS_GO
    TI_CHECK_LAUNCH("stream_step");
    return 0;
}
