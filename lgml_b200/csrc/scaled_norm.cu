// The seam between two layers whose results are scaled channel by channel before they join the residual stream:
//
//   x   <- keep x + s_a (ma A) + s_b (mb B)          A: a product's partial sums (and bias); B: rows of a tensor, or a token's
//                                                     rows among tiles of experts' outputs, added up
//   out  = x / sqrt(mean(x^2) + eps) * w             written row by row and, for a layer whose experts are known
//                                                     beforehand, also into the tiles of the experts that will read it
//
// or, without a norm, x as two bfloat16 rows (x rounded, and what the rounding lost), for a product that reads x itself.
// Everything is float32 but for the rows that feed a product.
#include <math.h>

#include "common.cuh"

LGML_DEFINE_LAST_ERROR(lgml_scaled_norm)

namespace {
struct Args {
    float *x;                   // [n, E]
    int keep;                   // 0: what x held is replaced
    const float *a;             // n_parts parts, a_stride floats apart, rows lda floats apart; null: none
    int n_parts, lda;
    long long a_stride, a_second;       // a_second: a row's second half lies this many floats further (0: none)
    const float *a_bias, *a_scale;      // [E] or null (null scale: ones)
    float a_mul;
    const float *b;             // rows ldb floats apart; null: none
    int ldb;
    const int *b_pos;           // null: row t; else the rows b_pos[t b_top ...] of token t
    int b_top;
    const float *b_scale;
    float b_mul;
    const int *rows;            // output row r is x's row rows[r] (x is then not written); null: row r
    const float *w;             // null: no norm
    float eps;
    void *out;                  // [rows, E]
    __nv_bfloat16 *tiles;       // the normed row again at rows tile_pos[t tile_top ...]; null: no
    const int *tile_pos;
    int tile_top;
    __nv_bfloat16 *split;       // without a norm: x rounded in rows 0 .. n - 1, the rest of x in rows n .. 2 n - 1; null: no
    int n, E, vec;
};

__device__ __forceinline__ void load4(const float *p, int i, int E, int vec, float (&v)[4]) {
    if (vec) {
        const float4 q = act_load(reinterpret_cast<const float4 *>(p + i));
        v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = i + e < E ? act_load(p + i + e) : 0.f;
    }
}
__device__ __forceinline__ void const4(const float *p, int i, int E, int vec, float (&v)[4]) {
    if (vec) {
        const float4 q = __ldg(reinterpret_cast<const float4 *>(p + i));
        v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = i + e < E ? __ldg(p + i + e) : 0.f;
    }
}
__device__ __forceinline__ void store4(float *p, int i, int E, int vec, const float (&v)[4]) {
    if (vec) {
        *reinterpret_cast<float4 *>(p + i) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (i + e < E) p[i + e] = v[e];
    }
}
__device__ __forceinline__ void store4(__nv_bfloat16 *p, int i, int E, int vec, const float (&v)[4]) {
    if (vec) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        *reinterpret_cast<uint2 *>(p + i) = make_uint2(*reinterpret_cast<unsigned *>(&lo), *reinterpret_cast<unsigned *>(&hi));
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (i + e < E) p[i + e] = __float2bfloat16_rn(v[e]);
    }
}

// A block a row; thread i holds the quads i, i + threads, ... of it (NQ of them).  The number of threads is the width's, so that a
// row's sums are formed in one order whatever else is in the batch (but for few bfloat16 rows, which get a thread a quad).
// PARTS: A comes in several parts (or halves): up to eight of them are in flight at a time.  Without them, for many rows, a
// thread needs few enough registers for two blocks or more an SM.
template <typename TO, int NQ, bool PARTS>
__global__ void __launch_bounds__(NQ > 4 || (NQ == 1 && PARTS) ? 1024 : 512, NQ > 2 || PARTS ? 1 : 2) scaled_norm_kernel(const Args a) {
    pdl_trigger();
    pdl_wait();
    __shared__ float red[32];
    const int r = blockIdx.x, E = a.E, T = blockDim.x;
    const size_t t = a.rows ? (size_t)a.rows[r] : (size_t)r;
    float *xr = a.x + t * E;
    constexpr bool AHEAD = NQ <= 4;         // very wide rows load as they go
    constexpr int ND = AHEAD ? NQ : 1;
    float v[NQ][4], da[ND][4], db[ND][4], dc[ND][4];
    const float *ar = a.a ? a.a + t * a.lda : nullptr;
    const float *br = nullptr, *cr = nullptr;           // B, and a token's second expert
    if (a.b) br = a.b + (a.b_pos ? (size_t)act_load(a.b_pos + t * a.b_top) : t) * a.ldb;
    if (a.b && a.b_pos && a.b_top > 1) cr = a.b + (size_t)act_load(a.b_pos + t * a.b_top + 1) * a.ldb;
    // the first loads of all of them before any is used
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
        const int i = 4 * (q * T + threadIdx.x);
        v[q][0] = v[q][1] = v[q][2] = v[q][3] = 0.f;
        if (i >= E) continue;
        if (a.keep) load4(xr, i, E, a.vec, v[q]);
        if (AHEAD && ar) load4(ar, i, E, a.vec, da[q % ND]);
        if (AHEAD && br) load4(br, i, E, a.vec, db[q % ND]);
        if (AHEAD && cr) load4(cr, i, E, a.vec, dc[q % ND]);
    }
    float ss = 0.f;
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
        const int i = 4 * (q * T + threadIdx.x);
        if (i >= E) continue;
        float s[4];
        float (&ad)[4] = da[q % ND], (&bd)[4] = db[q % ND], (&cd)[4] = dc[q % ND];
        if (!AHEAD && ar) load4(ar, i, E, a.vec, ad);
        if (!AHEAD && br) load4(br, i, E, a.vec, bd);
        if (!AHEAD && cr) load4(cr, i, E, a.vec, cd);
        if (ar) {
            if (PARTS) {
                // the other parts (a row's halves one after the other), added in their order
                constexpr int W = NQ > 4 ? 2 : (NQ == 1 ? 6 : 8);
                const int total = a.a_second ? 2 * a.n_parts : a.n_parts;
                for (int p = 1; p < total; p += W) {
                    float o[W][4];
#pragma unroll
                    for (int k = 0; k < W; ++k)
                        if (p + k < total) {
                            const int m = p + k;
                            load4(ar + (size_t)(m < a.n_parts ? m : m - a.n_parts) * a.a_stride + (m < a.n_parts ? 0 : a.a_second), i, E, a.vec, o[k]);
                        }
#pragma unroll
                    for (int k = 0; k < W; ++k)
                        if (p + k < total)
#pragma unroll
                            for (int e = 0; e < 4; ++e) ad[e] += o[k][e];
                }
            }
            if (a.a_bias) {
                const4(a.a_bias, i, E, a.vec, s);
#pragma unroll
                for (int e = 0; e < 4; ++e) ad[e] += s[e];
            }
            if (a.a_scale) {
                const4(a.a_scale, i, E, a.vec, s);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[q][e] = fmaf(ad[e] * a.a_mul, s[e], v[q][e]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[q][e] = fmaf(ad[e], a.a_mul, v[q][e]);
            }
        }
        if (br) {
            if (cr) {
#pragma unroll
                for (int e = 0; e < 4; ++e) bd[e] += cd[e];
            }
            if (a.b_pos)
                for (int k = 2; k < a.b_top; ++k) {
                    load4(a.b + (size_t)act_load(a.b_pos + t * a.b_top + k) * a.ldb, i, E, a.vec, s);
#pragma unroll
                    for (int e = 0; e < 4; ++e) bd[e] += s[e];
                }
            if (a.b_scale) {
                const4(a.b_scale, i, E, a.vec, s);
#pragma unroll
                for (int e = 0; e < 4; ++e) v[q][e] = fmaf(bd[e] * a.b_mul, s[e], v[q][e]);
            } else {
#pragma unroll
                for (int e = 0; e < 4; ++e) v[q][e] = fmaf(bd[e], a.b_mul, v[q][e]);
            }
        }
        if (!a.rows && (ar || br || !a.keep)) store4(xr, i, E, a.vec, v[q]);
        if (a.split) {
            float lo[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) lo[e] = v[q][e] - __bfloat162float(__float2bfloat16_rn(v[q][e]));
            store4(a.split + t * E, i, E, a.vec, v[q]);
            store4(a.split + ((size_t)a.n + t) * E, i, E, a.vec, lo);
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(v[q][e], v[q][e], ss);
    }
    if (!a.w) return;
    ss = block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)E + a.eps);
    TO *orow = reinterpret_cast<TO *>(a.out) + (size_t)r * E;
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
        const int i = 4 * (q * T + threadIdx.x);
        if (i >= E) continue;
        float w[4];
        const4(a.w, i, E, a.vec, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[q][e] = v[q][e] * inv * w[e];
        store4(orow, i, E, a.vec, v[q]);
        if (a.tiles)
            for (int k = 0; k < a.tile_top; ++k) store4(a.tiles + (size_t)act_load(a.tile_pos + t * a.tile_top + k) * E, i, E, a.vec, v[q]);
    }
}

template <typename TO>
int launch(const Args &a, int n_rows, cudaStream_t stream) {
    const int quads = (a.E + 3) / 4;
    auto threads = [&](int nq) { return ((quads + nq - 1) / nq + 31) / 32 * 32; };
    const bool parts = a.a != nullptr && (a.n_parts > 1 || a.a_second != 0);
#define LGML_SN(NQ)                                                                                              \
    do {                                                                                                         \
        if (parts) lgml_launch(scaled_norm_kernel<TO, NQ, true>, n_rows, threads(NQ), 0, stream, a);             \
        else lgml_launch(scaled_norm_kernel<TO, NQ, false>, n_rows, threads(NQ), 0, stream, a);                  \
    } while (0)
    if (quads <= 256) LGML_SN(1);
    else if (sizeof(TO) == 2 && parts && n_rows <= 64 && quads <= 1024) LGML_SN(1);      // few rows: a thread a quad (a decode step is latency)
    else if (quads <= 1024) LGML_SN(2);
    else if (quads <= 2048) LGML_SN(4);
    else if (quads <= 8192) LGML_SN(8);
    else LGML_FAIL("scaled_norm: rows of %d are too wide", a.E);
#undef LGML_SN
    return lgml_launch_status("scaled_norm");
}
}  // namespace

// x float32 [n, E].  n_rows: output rows (n without `rows`).  out_dtype: of `out`; tiles and split are bfloat16.
LGML_API int lgml_scaled_norm(float *x, int keep, const float *a, int n_parts, long long a_stride, int lda, long long a_second, const float *a_bias,
                              const float *a_scale, float a_mul, const float *b, int ldb, const int *b_pos, int b_top, const float *b_scale, float b_mul,
                              const int *rows, const float *w, float eps, void *out, int out_dtype, void *tiles, const int *tile_pos, int tile_top, void *split,
                              int n, int n_rows, int E, cudaStream_t stream) {
    LGML_REQUIRE(n >= 0 && n_rows >= 0 && E > 0 && n_parts >= 1, "scaled_norm: bad sizes");
    LGML_REQUIRE(rows != nullptr || n_rows == n, "scaled_norm: without a row list every row is an output row");
    LGML_REQUIRE((w == nullptr) == (out == nullptr), "scaled_norm: a norm has a weight and an output");
    LGML_REQUIRE(rows == nullptr || (split == nullptr && tiles == nullptr), "scaled_norm: listed rows go to the output only");
    LGML_REQUIRE(tiles == nullptr || (w != nullptr && tile_pos != nullptr && tile_top > 0 && out_dtype == LGML_BF16), "scaled_norm: tiles hold normed bfloat16 rows");
    LGML_REQUIRE(b_pos == nullptr || b_top > 0, "scaled_norm: bad number of experts' rows");
    if (n_rows == 0) return 0;
    Args p;
    p.x = x, p.keep = keep, p.a = a, p.n_parts = n_parts, p.lda = lda, p.a_stride = a_stride, p.a_second = a_second, p.a_bias = a_bias, p.a_scale = a_scale;
    p.a_mul = a_mul, p.b = b, p.ldb = ldb, p.b_pos = b_pos, p.b_top = b_top, p.b_scale = b_scale, p.b_mul = b_mul, p.rows = rows, p.w = w, p.eps = eps;
    p.out = out, p.tiles = (__nv_bfloat16 *)tiles, p.tile_pos = tile_pos, p.tile_top = tile_top, p.split = (__nv_bfloat16 *)split, p.n = n, p.E = E;
    p.vec = E % 4 == 0 && lda % 4 == 0 && ldb % 4 == 0 && a_stride % 4 == 0 && a_second % 4 == 0 &&
            (((uintptr_t)x | (uintptr_t)a | (uintptr_t)a_bias | (uintptr_t)a_scale | (uintptr_t)b | (uintptr_t)b_scale | (uintptr_t)w | (uintptr_t)out |
              (uintptr_t)tiles | (uintptr_t)split) & 15) == 0;
    if (out_dtype == LGML_F32) return launch<float>(p, n_rows, stream);
    if (out_dtype == LGML_BF16) return launch<__nv_bfloat16>(p, n_rows, stream);
    LGML_FAIL("scaled_norm: unknown type %d", out_dtype);
}
