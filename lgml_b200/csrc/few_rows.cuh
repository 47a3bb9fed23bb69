// Products of a handful of rows with a matrix, where the matrix is what has to be read: NT rows of x as
// floats in shared memory, and `lanes` neighbouring lanes of a warp (a power of two) on one row of the matrix, sixteen
// bytes a lane and turn, so that a warp's load covers whole lines of 32 / lanes rows.  Float32 sums in an order that
// depends on the row's length only.
#pragma once
#include "common.cuh"

template <typename T> struct RowPiece;
template <> struct RowPiece<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float *p, float (&v)[4]) {
        const float4 r = __ldg(reinterpret_cast<const float4 *>(p));
        v[0] = r.x, v[1] = r.y, v[2] = r.z, v[3] = r.w;
    }
};
template <> struct RowPiece<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16 *p, float (&v)[8]) {
        const uint4 r = __ldg(reinterpret_cast<const uint4 *>(p));
        const unsigned w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) v[2 * i] = __uint_as_float(w[i] << 16), v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
};

// lanes that share a row of K elements: the smallest power of two that covers it in one turn, at most 32
template <typename T> static inline int few_rows_lanes(int K) {
    int lanes = 1;
    while (lanes < 32 && lanes * RowPiece<T>::N < K) lanes *= 2;
    return lanes;
}
// may rows of K elements from `base` on be read in sixteen-byte pieces?
template <typename T> static inline bool few_rows_vec(const void *base, int K) {
    return K % RowPiece<T>::N == 0 && ((uintptr_t)base & 15) == 0;
}

// This lane's share of x_j . row for NT rows of x (xs, `ld` floats apart, 16-byte aligned, ld a multiple of 4; zeros where there is no row)
template <typename T, int NT>
__device__ __forceinline__ void few_rows_share(const T *row, const float *xs, int ld, int K, int sub, int lanes, bool vec, float (&acc)[NT]) {
    constexpr int V = RowPiece<T>::N;
    if (vec) {
        for (int k = sub * V; k < K; k += lanes * V) {
            float w[V];
            RowPiece<T>::load(row + k, w);
#pragma unroll
            for (int j = 0; j < NT; ++j) {
#pragma unroll
                for (int i = 0; i < V; i += 4) {
                    const float4 x = *reinterpret_cast<const float4 *>(xs + j * ld + k + i);
                    acc[j] = fmaf(x.x, w[i], fmaf(x.y, w[i + 1], fmaf(x.z, w[i + 2], fmaf(x.w, w[i + 3], acc[j]))));
                }
            }
        }
    } else {
        for (int k = sub; k < K; k += lanes) {
            const float w = to_f32(row[k]);
#pragma unroll
            for (int j = 0; j < NT; ++j) acc[j] = fmaf(xs[j * ld + k], w, acc[j]);
        }
    }
}

// the sum over the `lanes` lanes of a row, in every one of them
template <int NT> __device__ __forceinline__ void few_rows_reduce(float (&acc)[NT], int lanes) {
    for (int o = lanes >> 1; o > 0; o >>= 1) {
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[j] += __shfl_xor_sync(0xffffffffu, acc[j], o);
    }
}
