// A causal convolution over time of one channel (or of 16 bytes of neighbouring channels) at one token, and the step of
// its history. `hist` float32 [taps - 1][width]: the request's earlier inputs, oldest first; w float32 [taps][width], tap by
// tap (null: a plain sum of weight one, used with one tap); column `col` of rows of ld_in elements holds the inputs.
#pragma once
#include "common.cuh"

constexpr int SC_MAX_TAPS = 16;

template <typename T>
__device__ __forceinline__ float conv_at(const T* __restrict__ in, int ld_in, int col, int t, int local,
                                         const float* __restrict__ hist, int width, int c,
                                         const float* __restrict__ w, int taps) {
    float acc = 0.f;
    for (int j = 0; j < taps; ++j) {                       // column taps - 1 meets the current token
        const int back = taps - 1 - j;
        const float v = local - back >= 0 ? to_f32(in[(size_t)(t - back) * ld_in + col])
                                          : hist[(size_t)(taps - 1 + local - back) * width + c];
        acc = fmaf(w[(size_t)j * width + c], v, acc);
    }
    return acc;
}

// A step in which every request brings ONE token: the thread that made the token's output is the only one that
// read this channel's history, so it may also move the history on by one (oldest out, the token's input in).
__device__ __forceinline__ void conv_shift_history(float* __restrict__ hist, int width, int c, int taps, float newest) {
    float kept[SC_MAX_TAPS];
    for (int j = 1; j < taps - 1; ++j) kept[j] = hist[(size_t)j * width + c];
    for (int j = 1; j < taps - 1; ++j) hist[(size_t)(j - 1) * width + c] = kept[j];
    hist[(size_t)(taps - 2) * width + c] = newest;
}

// ------------------------------------------------------------------ sixteen bytes of channels a thread
template <typename T, int V>
__device__ __forceinline__ void load_row(const T* __restrict__ p, float* v) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = to_f32(e[i]);
}
template <typename T, int V>
__device__ __forceinline__ void store_row(T* __restrict__ p, const float* v) {
    uint4 raw;
    T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = from_f32<T>(v[i]);
    *reinterpret_cast<uint4*>(p) = raw;
}

// acc[i] = sum_j w[j][c0 + i] * in(t - (taps - 1 - j))[c0 + i]; newest[i]: the current token's own input.
template <typename T, int V>
__device__ __forceinline__ void conv_at_vec(const T* __restrict__ in, int ld_in, int col0, int t, int local,
                                            const float* __restrict__ hist, int width, int c0,
                                            const float* __restrict__ w, int taps, float* acc, float* newest) {
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = 0.f;
    for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;
        float v[V];
        if (local - back >= 0) {
            load_row<T, V>(in + (size_t)(t - back) * ld_in + col0, v);
        } else {
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = hist[(size_t)(taps - 1 + local - back) * width + c0 + i];
        }
        float wj[V];
        if (w) {
#pragma unroll
            for (int i = 0; i < V; i += 4) {
                const float4 f = *reinterpret_cast<const float4*>(w + (size_t)j * width + c0 + i);
                wj[i] = f.x; wj[i + 1] = f.y; wj[i + 2] = f.z; wj[i + 3] = f.w;
            }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] = fmaf(w ? wj[i] : 1.f, v[i], acc[i]);
        if (back == 0) {
#pragma unroll
            for (int i = 0; i < V; ++i) newest[i] = v[i];
        }
    }
}
