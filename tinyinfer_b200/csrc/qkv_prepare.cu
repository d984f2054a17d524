// Between the packed product [q | k | v] of an attention layer and its attention, all in one kernel, a block a token (in
// steps of few tokens several blocks a token, each with some of its heads):
//   convolution : optional short causal convolution per channel of q, k and v (short_conv.cuh; weights float32
//                 [taps][q | k | v], the earlier inputs in the request's state slot), before everything else
//   norm        : 0 none; 1 RMS norm over ALL rows of q, and of k, at once with a weight per row; 2 RMS norm per head with a
//                 weight per head feature; 3 per head AFTER the rotation, x / rms(x), with a weight or (null) without
//   rotation    : the first rotary_dim features of every head of q and k, in half-split or interleaved pairs, by angles from
//                 inverse frequencies or from a table. A token's cosines and sines are made once and serve all its heads
//   append      : k and v go to the token's place in its page, planes 2 (d == dv): [2][pages][Hkv][page][d], planes 1: rows
//                 [k (d) | v (dv)]; q goes to q_out [T][Hq][d]
// Float32 from the loads to the one rounding at each store. (head_rotation.cu does the per-head part alone, for rows of any
// layout; this kernel is for layers whose norm spans heads or whose rows are convolved first.)
#include "common.cuh"
#include "short_conv.cuh"

constexpr int QP_MAX_D = 512;

struct QkvPrepareArgs {
    void *q_out, *cache; int planes; long long v_plane_off;
    const void* in; int ld_in, in_off;
    const float* conv_w; float* hist; long long slot_stride; int taps, shift_history;
    int norm; const float *q_w, *k_w; float eps;
    const float *inv_freq, *table; int table_positions, interleaved, rotary_dim; float rot_factor;
    const int *positions, *token_seq, *cu_seqlens, *state_slots, *block_table; int max_blocks;
    int hq, hkv, d, dv, page_size, num_pages;
    int heads_per_block;          // of the token's hq + 2 hkv heads: q heads, then k heads, then v heads
    int* status;
};

template <int N> struct QpPack;
template <> struct QpPack<1> {
    static __device__ __forceinline__ void store(float* p, const float* v) { *p = v[0]; }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* v) { *p = __float2bfloat16_rn(v[0]); }
};
template <> struct QpPack<4> {
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

// VEC: neighbouring channels a thread loads at a time (16 bytes of them, or 1); HV: neighbouring features of a head a lane
// turns and stores at a time (4 or 1).
// PIECES: pieces of HV features of a head that a lane holds at most.
template <typename T, int VEC, int HV, int PIECES>
__global__ void __launch_bounds__(512) qkv_prepare_kernel(QkvPrepareArgs a) {
    extern __shared__ __align__(16) float qp_smem[];
    __shared__ float red[33];
    const int cq = a.hq * a.d, ck = a.hkv * a.d, width = cq + ck + a.hkv * a.dv;
    const int head0 = blockIdx.y * a.heads_per_block, head1 = min(a.hq + 2 * a.hkv, head0 + a.heads_per_block);
    auto channel_of = [&](int head) { return head <= a.hq + a.hkv ? head * a.d : cq + ck + (head - a.hq - a.hkv) * a.dv; };
    const int c_begin = channel_of(head0), c_end = channel_of(head1);    // the block's channels
    float* turn = qp_smem;                                    // [cosines | sines] of the token's position
    float* buf = qp_smem + ((a.rotary_dim + 3) & ~3);         // the block's share of [q | k], float32
    const int half = a.rotary_dim >> 1;
    ti_grid_launch_dependents();
    ti_grid_wait();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pos = a.positions[t], seq = a.token_seq[t];
    if (a.table != nullptr && (pos < 0 || pos >= a.table_positions)) {
        if (tid == 0 && a.status) atomicExch(a.status, 4);    // a position the table does not reach
        return;
    }
    const int logical = pos / a.page_size;
    const int page = logical < a.max_blocks ? a.block_table[(size_t)seq * a.max_blocks + logical] : -1;
    const bool has_page = page >= 0 && page < a.num_pages;
    if (!has_page && tid == 0 && a.status) atomicExch(a.status, 1);      // a token without a page: its k and v are not written
    const size_t place0 = has_page ? ((size_t)page * a.hkv) * a.page_size + pos % a.page_size : 0;
    const int row_len = a.planes == 2 ? a.d : a.d + a.dv;
    const long long v_off = a.planes == 2 ? a.v_plane_off : a.d;
    const int local = t - a.cu_seqlens[seq];
    float* hist = a.taps > 1 ? a.hist + (size_t)a.state_slots[seq] * a.slot_stride : nullptr;
    const T* in = (const T*)a.in;

    for (int j = tid; j < half; j += blockDim.x) {
        float s, c;
        if (a.table != nullptr) {
            c = a.table[(size_t)pos * a.rotary_dim + j];
            s = a.table[(size_t)pos * a.rotary_dim + half + j];
        } else {
            sincosf((float)pos * a.inv_freq[j], &s, &c);
        }
        turn[j] = c * a.rot_factor;
        turn[half + j] = s * a.rot_factor;
    }
    float ss_q = 0.f, ss_k = 0.f;
    for (int c0 = c_begin + tid * VEC; c0 < c_end; c0 += blockDim.x * VEC) {
        float v[VEC], newest[VEC];
        if constexpr (VEC == 1) {
            newest[0] = to_f32(in[(size_t)t * a.ld_in + a.in_off + c0]);
            v[0] = a.taps > 1 ? conv_at(in, a.ld_in, a.in_off + c0, t, local, (const float*)hist, width, c0, a.conv_w, a.taps)
                              : (a.conv_w ? a.conv_w[c0] : 1.f) * newest[0];
        } else {
            conv_at_vec<T, VEC>(in, a.ld_in, a.in_off + c0, t, local, hist, width, c0, a.conv_w, a.taps, v, newest);
        }
        if (a.shift_history && a.taps > 1) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) conv_shift_history(hist, width, c0 + e, a.taps, newest[e]);
        }
        if (c0 >= cq + ck) {
            if (has_page) {
                const int head = (c0 - cq - ck) / a.dv, f = (c0 - cq - ck) % a.dv;
                T* dst = (T*)a.cache + (place0 + (size_t)head * a.page_size) * row_len + v_off + f;
                if constexpr (VEC == 1) *dst = from_f32<T>(v[0]);
                else store_row<T, VEC>(dst, v);
            }
            continue;
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            buf[c0 - c_begin + e] = v[e];
            if (c0 < cq) ss_q = fmaf(v[e], v[e], ss_q);
            else ss_k = fmaf(v[e], v[e], ss_k);
        }
    }
    float inv_q = 1.f, inv_k = 1.f;
    if (a.norm == 1) {
        inv_q = rsqrtf(block_sum(ss_q, red) / (float)cq + a.eps);
        inv_k = rsqrtf(block_sum(ss_k, red) / (float)ck + a.eps);
    }
    __syncthreads();

    const int warps = blockDim.x >> 5;
    for (int head = head0 + warp; head < min(head1, a.hq + a.hkv); head += warps) {
        const bool is_q = head < a.hq;
        float* x = buf + (size_t)(head - head0) * a.d;        // q heads, then k heads
        const float* w = is_q ? a.q_w : a.k_w;
        if (a.norm == 1 || a.norm == 2) {                     // each lane scales its own features; a partner is read below
            float inv = is_q ? inv_q : inv_k;
            const float* wh = w + (a.norm == 1 ? (size_t)(is_q ? head : head - a.hq) * a.d : 0);
            if (a.norm == 2) {
                float ss = 0.f;
                for (int i = lane; i < a.d; i += 32) ss = fmaf(x[i], x[i], ss);
                inv = rsqrtf(warp_sum(ss) / (float)a.d + a.eps);
            }
            for (int i = lane; i < a.d; i += 32) x[i] = wh[i] * x[i] * inv;
            __syncwarp();
        }
        float y[PIECES][HV];
        float ss = 0.f;
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int i0 = (p * 32 + lane) * HV;
            if (i0 >= a.d) break;
#pragma unroll
            for (int e = 0; e < HV; ++e) {
                const int i = i0 + e;
                float o = x[i];
                if (i < a.rotary_dim) {
                    const int j = a.interleaved ? i >> 1 : (i < half ? i : i - half);
                    const int other = a.interleaved ? i ^ 1 : (i < half ? i + half : i - half);
                    const bool leads = a.interleaved ? !(i & 1) : i < half;
                    const float c = turn[j], s = turn[half + j];
                    o = leads ? o * c - x[other] * s : o * c + x[other] * s;
                }
                y[p][e] = o;
                ss = fmaf(o, o, ss);
            }
        }
        float inv = 1.f;
        if (a.norm == 3) inv = rsqrtf(warp_sum(ss) / (float)a.d + a.eps);
        T* dst;
        if (is_q) dst = (T*)a.q_out + (size_t)t * cq + (size_t)head * a.d;
        else if (has_page) dst = (T*)a.cache + (place0 + (size_t)(head - a.hq) * a.page_size) * row_len;
        else continue;
#pragma unroll
        for (int p = 0; p < PIECES; ++p) {
            const int i0 = (p * 32 + lane) * HV;
            if (i0 >= a.d) break;
            if (a.norm == 3) {
#pragma unroll
                for (int e = 0; e < HV; ++e) y[p][e] *= w != nullptr ? w[i0 + e] * inv : inv;
            }
            QpPack<HV>::store(dst + i0, y[p]);
        }
    }
}

// norm: see the head of the file. conv_w float32 [taps][width] over the packed channels (null with taps 1: no convolution);
// hist: the requests' state slots, [taps - 1][width] each, slot_stride floats apart; shift_history: every request of the
// step brings one token and the kernel also moves the histories on (otherwise ti_conv_state_update does, afterwards). The
// packed rows are columns [in_off, in_off + width) of rows of ld_in elements.
TI_API int ti_qkv_prepare(void* q_out, void* cache, int planes, const void* in, int ld_in, int in_off, const float* conv_w,
                          float* hist, long long slot_stride, int taps, int shift_history, int norm, const float* q_w,
                          const float* k_w, float eps, const float* inv_freq, const float* cos_sin_table, int table_positions,
                          int interleaved, int rotary_dim, float rot_factor, const int* positions, const int* token_seq,
                          const int* cu_seqlens, const int* state_slots, const int* block_table, int max_blocks, int num_tokens,
                          int hq, int hkv, int d, int dv, int page_size, int num_pages, int* status, int dtype,
                          cudaStream_t stream) {
    TI_REQUIRE(num_tokens >= 0 && hq > 0 && hkv > 0 && d > 0 && d <= QP_MAX_D && dv > 0 && page_size > 0 && num_pages > 0,
               "qkv_prepare: bad sizes (heads of at most %d features)", QP_MAX_D);
    TI_REQUIRE(rotary_dim >= 0 && rotary_dim <= d && rotary_dim % 2 == 0,
               "qkv_prepare: rotary_dim %d must be even and at most the head size %d", rotary_dim, d);
    TI_REQUIRE(rotary_dim == 0 || (inv_freq == nullptr) != (cos_sin_table == nullptr),
               "qkv_prepare: a rotation comes from inverse frequencies or from a table");
    TI_REQUIRE(cos_sin_table == nullptr || table_positions > 0, "qkv_prepare: a table needs its number of positions");
    TI_REQUIRE(norm >= 0 && norm <= 3 && ((norm != 1 && norm != 2) || (q_w && k_w)), "qkv_prepare: norm %d lacks its weights", norm);
    TI_REQUIRE(taps >= 1 && taps <= SC_MAX_TAPS && (taps == 1 || (conv_w && hist)),
               "qkv_prepare: a convolution (1..%d taps) needs its weights and the history", SC_MAX_TAPS);
    TI_REQUIRE(cache && block_table && (planes == 1 || (planes == 2 && d == dv)),
               "qkv_prepare: a cache of two planes needs keys and values of one size");
    const int cq = hq * d, ck = hkv * d, width = cq + ck + hkv * dv;
    TI_REQUIRE(in_off >= 0 && ld_in >= in_off + width, "qkv_prepare: the packed rows do not fit their tensor's rows");
    if (num_tokens == 0) return 0;
    QkvPrepareArgs a = {q_out, cache, planes, (long long)num_pages * hkv * page_size * d, in, ld_in, in_off, conv_w, hist,
                        slot_stride, taps, shift_history ? 1 : 0, norm, q_w, k_w, eps, inv_freq, cos_sin_table, table_positions,
                        interleaved, rotary_dim, rot_factor, positions, token_seq, cu_seqlens, state_slots, block_table,
                        max_blocks, hq, hkv, d, dv, page_size, num_pages, hq + 2 * hkv, status};
    const size_t smem = (size_t)(cq + ck + ((rotary_dim + 3) & ~3)) * sizeof(float);
    TI_REQUIRE(smem <= 200 * 1024, "qkv_prepare: %d rows of q and k do not fit shared memory", cq + ck);
    const int vec = dtype == TI_F32 ? 4 : 8;
    // (few tokens with a history: a channel a thread, so that many threads read it side by side)
    const bool wide = (taps == 1 || num_tokens > 128) && d % vec == 0 && dv % vec == 0 && ld_in % vec == 0 && in_off % vec == 0 &&
                      ((uintptr_t)q_out | (uintptr_t)cache | (uintptr_t)in | (uintptr_t)conv_w) % 16 == 0;
    const bool heads4 = d % 4 == 0 && dv % 4 == 0 && ((uintptr_t)q_out | (uintptr_t)cache) % 16 == 0;
    // few tokens: every channel group of a token at once; many: blocks enough to fill the machine anyway
    // a token's heads over several blocks, unless the norm spans them
    const int heads = hq + 2 * hkv;
    int splits = 1;
    if (norm != 1)
        while (splits * 2 <= heads && splits * 2 * num_tokens <= 148) splits <<= 1;
    a.heads_per_block = (heads + splits - 1) / splits;
    splits = (heads + a.heads_per_block - 1) / a.heads_per_block;
    const int share = splits > 1 ? a.heads_per_block * (d > dv ? d : dv) : width;
    int threads = 128;
    const int most = num_tokens <= 2 * 148 ? 512 : 256;
    while (threads < most && threads * (wide ? vec : 1) < share) threads <<= 1;
    typedef __nv_bfloat16 B;
#define QP_GO(T, V, H)                                                                                                       \
    do {                                                                                                                     \
        if (d <= 32 * (H)) QP_GO_P(T, V, H, 1);                                                                              \
        else QP_GO_P(T, V, H, QP_MAX_D / (32 * (H)));                                                                        \
    } while (0)
#define QP_GO_P(T, V, H, P)                                                                                                     \
    do {                                                                                                                     \
        if (smem > 40 * 1024) {                                                                                              \
            const cudaError_t e = cudaFuncSetAttribute(qkv_prepare_kernel<T, V, H, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, \
                                                       (int)smem);                                                           \
            TI_REQUIRE(e == cudaSuccess, "qkv_prepare: shared memory: %s", cudaGetErrorString(e));                           \
        }                                                                                                                    \
        ti_launch(qkv_prepare_kernel<T, V, H, P>, dim3(num_tokens, splits), threads, smem, stream, a);                                        \
    } while (0)
    if (dtype == TI_F32) { if (wide) QP_GO(float, 4, 4); else if (heads4) QP_GO(float, 1, 4); else QP_GO(float, 1, 1); }
    else if (dtype == TI_BF16) { if (wide) QP_GO(B, 8, 4); else if (heads4) QP_GO(B, 1, 4); else QP_GO(B, 1, 1); }
    else TI_REQUIRE(false, "qkv_prepare: unknown dtype %d", dtype);
#undef QP_GO
#undef QP_GO_P
    TI_CHECK_LAUNCH("qkv_prepare");
    return 0;
}
