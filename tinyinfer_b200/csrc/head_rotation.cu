// Per-head norm and rotary rotation of packed rows [q | k | v] whose pieces may differ in size, for mixers that
// are not served by the fused kernel of the plain decoder (rope_append.cu): keys and values of different sizes,
// rows that hold more than q, k and v, layers that only have queries, and mixers that keep no pages at all.
//   in  : rows of ld_in elements, first column in_off: Hq heads of d query features, then (has_kv) Hkv heads of d key
//         features and Hkv heads of dv value features
//   q, k: optional RMS norm over the head with a plain weight, then the rotation of the first rotary_dim features
//         (same rotation data as rope_append.cu: inverse frequencies or a table of cosines and sines, half-split or
//         interleaved pairs; rot_factor multiplies every cosine and sine), then a constant factor (q_scale, k_scale);
//         v passes unchanged. norm_after != 0: the RMS norm comes AFTER the rotation instead, with the weight or, if
//         there is none, without one (x / rms(x))
//   out : q goes to out[t][head * d] (rows of ld_out). With a cache, k and v go to the token's place in its page:
//         planes 2 (d == dv): [2][pages][Hkv][page][d]; planes 1: rows [k (d) | v (dv)]. Without a cache and with
//         has_kv, k and v follow q in the row of out: [q | k | v], so that a recurrent mixer reads them from there.
//         A head of q and k may hold `maps` maps of d features side by side (differential attention): norm and rotation
//         are each map's own, and the maps of a key head lie side by side in its cache row (maps d features).
//         v_is_k: the values are the keys as they come, before norm and rotation; the rows hold no columns for them.
// Two kernels. Heads of a power of two of eight-feature pieces (8, 16, ... 256 features) whose rows lie on 16-byte boundaries:
// a block a token, eight neighbouring features a thread, all loads 16 bytes, a head's sum and a feature's partner by shuffles
// among the threads of its head, the token's cosines and sines made once for all its heads. Anything else: one warp a (token,
// head, map) through shared memory. Float32 arithmetic, one rounding at the store. OutT may be float32 for a bfloat16 input:
// what enters a float32 recurrence is then never rounded after its rotation.
#include "common.cuh"

constexpr int HR_WARPS = 4;
constexpr int HR_MAX_D = 512;

struct HeadRotationArgs {
    void* out; int ld_out;
    void* cache; int planes; long long v_plane_off;
    const void* in; int ld_in, in_off;
    const float *q_w, *k_w; float eps;
    const float *inv_freq, *table; int table_positions, interleaved, rotary_dim;
    float q_scale, k_scale, rot_factor; int norm_after;
    const int *positions, *token_seq, *block_table; int max_blocks;
    int hq, hkv, d, dv, has_kv, page_size, num_pages;       // hq, hkv: maps of query and of key heads
    int maps, v_is_k;
    int* status;
};

template <typename T, typename OutT>
__global__ void __launch_bounds__(HR_WARPS * 32) head_rotation_kernel(HeadRotationArgs a) {
    __shared__ float buf[HR_WARPS][HR_MAX_D];
    __shared__ float turned[HR_WARPS][HR_MAX_D];
    ti_grid_launch_dependents();
    ti_grid_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.x * HR_WARPS + warp;
    const int t = blockIdx.y;
    const int heads_total = a.hq + (a.has_kv ? a.hkv + a.hkv / a.maps : 0);
    if (head >= heads_total) return;
    const bool is_q = head < a.hq;
    const bool is_k = !is_q && head < a.hq + a.hkv;
    const int size = (is_q || is_k) ? a.d : a.dv;
    const int col = is_q ? head * a.d : is_k ? a.hq * a.d + (head - a.hq) * a.d
                                             : (a.hq + a.hkv) * a.d + (head - a.hq - a.hkv) * a.dv;
    const int from = (a.v_is_k && !is_q && !is_k) ? (head - a.hkv) * a.d : col;      // the key head of the same number
    const T* src = (const T*)a.in + (size_t)t * a.ld_in + a.in_off + from;
    float* x = buf[warp];
    float ss = 0.f;
    for (int i = lane; i < size; i += 32) {
        const float v = to_f32(src[i]);
        x[i] = v;
        ss += v * v;
    }
    const float* w = is_q ? a.q_w : (is_k ? a.k_w : nullptr);
    const bool norm_last = a.norm_after && (is_q || is_k);
    if (w != nullptr && !norm_last) {
        ss = warp_sum(ss);
        const float inv = rsqrtf(ss / (float)size + a.eps);
        for (int i = lane; i < size; i += 32) x[i] = w[i] * x[i] * inv;
    }
    __syncwarp();
    const int pos = a.positions[t];
    const bool rotate = (is_q || is_k) && (a.inv_freq != nullptr || a.table != nullptr) && a.rotary_dim > 0;
    if (rotate && a.table != nullptr && (pos < 0 || pos >= a.table_positions)) {
        if (lane == 0 && a.status) atomicExch(a.status, 4);          // a position the table does not reach
        return;
    }
    const float factor = is_q ? a.q_scale : is_k ? a.k_scale : 1.f;
    T* cdst = nullptr;
    OutT* odst = nullptr;
    if (is_q || a.cache == nullptr) {
        odst = (OutT*)a.out + (size_t)t * a.ld_out + col;
    } else {
        const int logical = pos / a.page_size;
        const int page = logical < a.max_blocks ? a.block_table[(size_t)a.token_seq[t] * a.max_blocks + logical] : -1;
        if (page < 0 || page >= a.num_pages) {
            if (lane == 0 && a.status) atomicExch(a.status, 1);      // a token without a page: never write
            return;
        }
        const int kvh = is_k ? (head - a.hq) / a.maps : head - a.hq - a.hkv;
        const int kd = a.maps * a.d, at = is_k ? (head - a.hq) % a.maps * a.d : 0;
        const size_t place = ((size_t)page * (a.hkv / a.maps) + kvh) * a.page_size + pos % a.page_size;
        if (a.planes == 2) cdst = (T*)a.cache + (is_k ? at : a.v_plane_off) + place * kd;
        else cdst = (T*)a.cache + place * (kd + a.dv) + (is_k ? at : kd);
    }
    const int half = a.rotary_dim >> 1;
    const float pos_f = (float)pos;
    float* y = turned[warp];
    float ss_after = 0.f;
    for (int i = lane; i < size; i += 32) {
        float o = x[i];
        if (rotate && i < a.rotary_dim) {
            const int j = a.interleaved ? (i >> 1) : (i < half ? i : i - half);
            const bool first = a.interleaved ? !(i & 1) : i < half;
            const int other = a.interleaved ? (i ^ 1) : (i < half ? i + half : i - half);
            float s, c;
            if (a.table != nullptr) {
                c = a.table[(size_t)pos * a.rotary_dim + j];
                s = a.table[(size_t)pos * a.rotary_dim + half + j];
            } else {
                sincosf(pos_f * a.inv_freq[j], &s, &c);
            }
            c *= a.rot_factor;
            s *= a.rot_factor;
            o = first ? x[i] * c - x[other] * s : x[i] * c + x[other] * s;
        }
        y[i] = o;                                   // read back by this lane alone
        ss_after += o * o;
    }
    float inv_after = 1.f;
    if (norm_last) inv_after = rsqrtf(warp_sum(ss_after) / (float)size + a.eps);
    for (int i = lane; i < size; i += 32) {
        float o = y[i];
        if (norm_last) o = (w != nullptr ? w[i] : 1.f) * o * inv_after;
        o *= factor;
        if (cdst) cdst[i] = from_f32<T>(o);
        else odst[i] = from_f32<OutT>(o);
    }
}

// ------------------------------------------------------------------ a block a token, eight features a thread
constexpr int HV_THREADS = 256;
constexpr int HV_MAX_ROTARY = 256;

__device__ __forceinline__ void hv_load(const __nv_bfloat16* p, float* v) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 f = __bfloat1622float2(b[i]);
        v[2 * i] = f.x;
        v[2 * i + 1] = f.y;
    }
}
__device__ __forceinline__ void hv_load(const float* p, float* v) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const float4 f = reinterpret_cast<const float4*>(p)[i];
        v[4 * i] = f.x; v[4 * i + 1] = f.y; v[4 * i + 2] = f.z; v[4 * i + 3] = f.w;
    }
}
__device__ __forceinline__ void hv_store(__nv_bfloat16* p, const float* v) {
    uint4 u;
    __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    *reinterpret_cast<uint4*>(p) = u;
}
__device__ __forceinline__ void hv_store(float* p, const float* v) {
#pragma unroll
    for (int i = 0; i < 2; ++i) reinterpret_cast<float4*>(p)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
}

// blockIdx.x: token; blockIdx.y: its share of the row's pieces (a multiple of a warp's) in steps of few tokens.
template <typename T, typename OutT>
__global__ void __launch_bounds__(HV_THREADS) head_rotation_vec_kernel(HeadRotationArgs a, int pieces_per_block) {
    __shared__ float turn[HV_MAX_ROTARY];                      // [cosines | sines] of the token's position
    ti_grid_launch_dependents();
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
    const int pos = a.positions[t];                            // an input of the step, not of the kernels before
    const bool turns = (a.inv_freq != nullptr || a.table != nullptr) && a.rotary_dim > 0;
    const int half = a.rotary_dim >> 1;
    if (turns && a.table != nullptr && (pos < 0 || pos >= a.table_positions)) {
        if (tid == 0 && a.status) atomicExch(a.status, 4);     // a position the table does not reach
        return;
    }
    if (turns) {
        for (int j = tid; j < half; j += HV_THREADS) {
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
    }
    const int group = a.d >> 3;                                // threads a head (map): a power of two, at most a warp
    const int nq = a.hq * group, nk = a.has_kv ? a.hkv * group : 0;
    const int vpieces = a.dv >> 3, kv_heads = a.hkv / a.maps;
    const int total = nq + nk + (a.has_kv ? kv_heads * vpieces : 0);
    const int first = blockIdx.y * pieces_per_block, last = min(total, first + pieces_per_block);
    size_t place0 = 0;                                         // the token's row of its page's first head
    bool has_page = true;
    if (a.cache != nullptr) {
        const int logical = pos / a.page_size;
        const int page = logical < a.max_blocks ? a.block_table[(size_t)a.token_seq[t] * a.max_blocks + logical] : -1;
        has_page = page >= 0 && page < a.num_pages;
        if (!has_page && tid == 0 && a.status) atomicExch(a.status, 1);      // a token without a page: its k and v are not written
        if (has_page) place0 = (size_t)page * kv_heads * a.page_size + pos % a.page_size;
    }
    const int kd = a.maps * a.d, row_len = a.planes == 2 ? kd : kd + a.dv;
    const long long v_at = a.planes == 2 ? a.v_plane_off : kd;
    __syncthreads();
    ti_grid_wait();
    const T* row = (const T*)a.in + (size_t)t * a.ld_in + a.in_off;
    for (int base = first; base < last; base += HV_THREADS) {  // whole warps go round together
        const int piece = base + tid;
        const bool real = piece < last;
        const bool is_q = piece < nq, is_k = !is_q && piece < nq + nk, is_v = !is_q && !is_k;
        float x[8] = {};
        if (real) {
            const int col = !is_v || !a.v_is_k ? piece : piece - nk;          // values that are the keys: the same columns
            hv_load(row + (size_t)col * 8, x);
        }
        const float* w = is_q ? a.q_w : is_k ? a.k_w : nullptr;
        const int i0 = (piece & (group - 1)) * 8;              // of a query or key head: the piece's first feature
        const bool normed = (is_q || is_k) && (w != nullptr || a.norm_after);
        float wv[8];
        if (w != nullptr) {
#pragma unroll
            for (int e = 0; e < 8; ++e) wv[e] = w[i0 + e];
        }
        auto norm = [&]() {                                    // all lanes; a head's pieces lie side by side in the warp
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(x[e], x[e], ss);
            for (int o = group >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if (normed) {
                const float inv = rsqrtf(ss / (float)a.d + a.eps);
#pragma unroll
                for (int e = 0; e < 8; ++e) x[e] = (w != nullptr ? wv[e] : 1.f) * x[e] * inv;
            }
        };
        const bool norms = a.q_w != nullptr || a.k_w != nullptr || a.norm_after;       // the same for the whole grid
        if (norms && !a.norm_after) norm();
        if (turns) {
            if (a.interleaved) {
                if (!is_v && i0 < a.rotary_dim) {
#pragma unroll
                    for (int e = 0; e < 8; e += 2) {
                        const float c = turn[(i0 + e) >> 1], s = turn[half + ((i0 + e) >> 1)];
                        const float u = x[e], v = x[e + 1];
                        x[e] = u * c - v * s;
                        x[e + 1] = v * c + u * s;
                    }
                }
            } else {
                const int hop = half >> 3;                     // the partner's pieces lie so many threads away
                const bool leads = i0 < half;
                const int from = !is_v && i0 < a.rotary_dim ? (leads ? lane + hop : lane - hop) : lane;
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float other = __shfl_sync(0xffffffffu, x[e], from);
                    if (!is_v && i0 < a.rotary_dim) {
                        const int j = (leads ? i0 : i0 - half) + e;
                        x[e] = leads ? x[e] * turn[j] - other * turn[half + j] : x[e] * turn[j] + other * turn[half + j];
                    }
                }
            }
        }
        if (norms && a.norm_after) norm();
        if (!real) continue;
        if (!is_v) {
            const float f = is_q ? a.q_scale : a.k_scale;
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= f;
        }
        if (is_q || a.cache == nullptr) {
            hv_store((OutT*)a.out + (size_t)t * a.ld_out + (size_t)piece * 8, x);
        } else if (has_page) {
            int head, at;                                      // the key or value head, and the piece's place in its cache row
            long long plane = 0;
            if (is_k) {
                const int map = (piece - nq) / group;
                head = map / a.maps;
                at = map % a.maps * a.d + i0;
            } else {
                head = (piece - nq - nk) / vpieces;
                at = (piece - nq - nk) % vpieces * 8;
                plane = v_at;
            }
            hv_store((T*)a.cache + plane + (place0 + (size_t)head * a.page_size) * row_len + at, x);
        }
    }
}

// hq, hkv: heads (of maps d features each); dtype: of `in` and of the cache; out_f32 != 0: `out` is float32 whatever the dtype.
TI_API int ti_head_rotation(void* out, int ld_out, void* cache, int planes, const void* in, int ld_in, int in_off,
                            const float* q_norm_w, const float* k_norm_w, float eps, const float* inv_freq,
                            const float* cos_sin_table, int table_positions, int interleaved, int rotary_dim, float rot_factor, float q_scale,
                            float k_scale, const int* positions, const int* token_seq, const int* block_table,
                            int max_blocks, int num_tokens, int hq, int hkv, int d, int dv, int has_kv, int page_size,
                            int num_pages, int maps, int v_is_k, int* status, int out_f32, int norm_after, int dtype, cudaStream_t stream) {
    TI_REQUIRE(maps >= 1 && (!v_is_k || (maps == 1 && d == dv && cache)), "head_rotation: values that are the keys come with one map, "
               "one size and a cache");
    TI_REQUIRE(d > 0 && d <= HR_MAX_D && dv > 0 && dv <= HR_MAX_D, "head_rotation: head sizes %d / %d not in 1..%d", d, dv, HR_MAX_D);
    TI_REQUIRE(rotary_dim >= 0 && rotary_dim <= d && rotary_dim % 2 == 0,
               "head_rotation: rotary_dim %d must be even and at most the head size %d", rotary_dim, d);
    TI_REQUIRE(hq > 0 && hkv >= 0 && num_tokens >= 0, "head_rotation: bad sizes");
    TI_REQUIRE(inv_freq == nullptr || cos_sin_table == nullptr, "head_rotation: inverse frequencies or a table, not both");
    TI_REQUIRE(cos_sin_table == nullptr || table_positions > 0, "head_rotation: a table needs its number of positions");
    TI_REQUIRE(cache == nullptr || (has_kv && (planes == 1 || (planes == 2 && maps * d == dv)) && page_size > 0 && block_table),
               "head_rotation: a cache of two planes needs keys and values of one size");
    TI_REQUIRE(num_tokens <= 65535, "head_rotation: more than 65535 tokens in one step");
    if (num_tokens == 0) return 0;
    HeadRotationArgs a = {out, ld_out, cache, planes, (long long)num_pages * hkv * page_size * maps * d, in, ld_in, in_off,
                          q_norm_w, k_norm_w, eps, inv_freq, cos_sin_table, table_positions, interleaved, rotary_dim,
                          q_scale, k_scale, rot_factor, norm_after ? 1 : 0, positions, token_seq, block_table, max_blocks, hq * maps, hkv * maps, d, dv, has_kv ? 1 : 0,
                          page_size, num_pages, maps, v_is_k ? 1 : 0, status};
    const int group = d / 8;
    const bool wide = d % 8 == 0 && group <= 32 && (group & (group - 1)) == 0 && (!has_kv || dv % 8 == 0) && rotary_dim <= HV_MAX_ROTARY &&
                      rotary_dim % (interleaved ? 8 : 16) == 0 && ld_in % 8 == 0 && in_off % 8 == 0 && ld_out % 8 == 0 &&
                      (((uintptr_t)out | (uintptr_t)in | (uintptr_t)cache) & 15) == 0;
    if (wide) {
        const int pieces = (hq * maps + (has_kv ? hkv * maps : 0)) * group + (has_kv ? hkv * (dv / 8) : 0);
        // few tokens: a token's pieces over several blocks, so that as many SMs work
        int shares = num_tokens >= 148 ? 1 : (pieces + HV_THREADS - 1) / HV_THREADS;
        const int per_block = shares == 1 ? pieces : HV_THREADS;
        dim3 grid(num_tokens, shares);
        if (dtype == TI_F32) ti_launch(head_rotation_vec_kernel<float, float>, grid, HV_THREADS, 0, stream, a, per_block);
        else if (dtype == TI_BF16 && out_f32) ti_launch(head_rotation_vec_kernel<__nv_bfloat16, float>, grid, HV_THREADS, 0, stream, a, per_block);
        else if (dtype == TI_BF16) ti_launch(head_rotation_vec_kernel<__nv_bfloat16, __nv_bfloat16>, grid, HV_THREADS, 0, stream, a, per_block);
        else TI_REQUIRE(false, "head_rotation: unknown dtype %d", dtype);
        TI_CHECK_LAUNCH("head_rotation");
        return 0;
    }
    const int heads_total = hq * maps + (has_kv ? hkv * maps + hkv : 0);
    dim3 grid((heads_total + HR_WARPS - 1) / HR_WARPS, num_tokens);
    if (dtype == TI_F32) ti_launch(head_rotation_kernel<float, float>, grid, HR_WARPS * 32, 0, stream, a);
    else if (dtype == TI_BF16 && out_f32) ti_launch(head_rotation_kernel<__nv_bfloat16, float>, grid, HR_WARPS * 32, 0, stream, a);
    else if (dtype == TI_BF16) ti_launch(head_rotation_kernel<__nv_bfloat16, __nv_bfloat16>, grid, HR_WARPS * 32, 0, stream, a);
    else TI_REQUIRE(false, "head_rotation: unknown dtype %d", dtype);
    TI_CHECK_LAUNCH("head_rotation");
    return 0;
}
