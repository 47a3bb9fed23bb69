// The residual stream as R parallel streams ("hyper-connections"), the gate on what a sublayer adds, and
// the RMS norm of what the next sublayer reads, in one pass over a token's streams:
//
//   z    = d [* sigmoid(gate)]                      d: a sublayer's result (a tensor or a product's partial sums + bias)
//   x_t  = sum_s mix[s, t] x_s + w_out[t] z         all streams at once from the old ones (no d: they stay as they are)
//   u    = sum_s w_in[s] x_s                        (w_in null: the plain sum)
//   out  = u / sqrt(mean(u^2) + eps) * w
//
// With `start` the streams do not exist yet: every x_s is the token's row of `start` times `start_scale`
// (then nothing is pending), and this kernel writes them.  Everything is float32; out is in the compute type.
#include <math.h>

#include "common.cuh"

LGML_DEFINE_LAST_ERROR(lgml_streams)

namespace {

constexpr int MAX_STREAMS = 8;

struct StreamArgs {
    float *x;                       // [n, R, E]
    const float *start;             // [n, E] or null
    float start_scale;
    const float *d;                 // [n_parts][n, E] or null
    int n_parts;
    long long part_stride;
    const float *d_bias;            // [E] or null
    const float *gate;              // [n, ldg] or null: before the sigmoid
    int ldg;
    const float *w_out, *mix;       // [R], [R, R] (from, to)
    const float *w_in;              // [R] or null
    const float *w;                 // [E] or null: no norm
    const int *rows;                // or null: the token rows to norm; the streams are then not written
    void *out;                      // [n_out, E]
    int E, R;
    float eps;
};

template <int V> struct Vec;
template <> struct Vec<1> {
    static __device__ __forceinline__ void load(const float *p, float (&v)[1]) { v[0] = act_load(p); }
    static __device__ __forceinline__ void load_w(const float *p, float (&v)[1]) { v[0] = __ldg(p); }
    static __device__ __forceinline__ void store(float *p, const float (&v)[1]) { p[0] = v[0]; }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, const float (&v)[1]) { p[0] = __float2bfloat16_rn(v[0]); }
};
template <> struct Vec<4> {
    static __device__ __forceinline__ void load(const float *p, float (&v)[4]) {
        const float4 t = act_load(reinterpret_cast<const float4 *>(p));
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    }
    static __device__ __forceinline__ void load_w(const float *p, float (&v)[4]) {
        const float4 t = __ldg(reinterpret_cast<const float4 *>(p));
        v[0] = t.x, v[1] = t.y, v[2] = t.z, v[3] = t.w;
    }
    static __device__ __forceinline__ void store(float *p, const float (&v)[4]) { *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]); }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, const float (&v)[4]) {
        __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
        float2 raw;
        raw.x = *reinterpret_cast<float *>(&lo), raw.y = *reinterpret_cast<float *>(&hi);
        *reinterpret_cast<float2 *>(p) = raw;
    }
};

// A block per row.  RT: the streams at compile time (MAX_STREAMS: any number up to it, tested at run time).
template <typename TO, int RT, int V>
__global__ void __launch_bounds__(512) stream_norm_kernel(const StreamArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float us[];        // u of the row
    __shared__ float red[32];
    using X = Vec<V>;
    const int E = a.E, r = blockIdx.x, R = RT == MAX_STREAMS ? a.R : RT;
    const size_t t = a.rows ? (size_t)a.rows[r] : (size_t)r;
    float *xr = a.x + t * (size_t)R * E;
    const bool has_d = a.d != nullptr;
    const bool write = a.rows == nullptr && (has_d || a.start != nullptr);
    float win[RT], wout[RT], mix[RT][RT];
#pragma unroll
    for (int s = 0; s < RT; ++s) {
        const bool on = s < R;
        win[s] = on ? (a.w_in ? __ldg(a.w_in + s) : 1.f) : 0.f;
        wout[s] = on && has_d ? __ldg(a.w_out + s) : 0.f;
#pragma unroll
        for (int q = 0; q < RT; ++q) mix[s][q] = on && q < R && has_d ? __ldg(a.mix + s * R + q) : 0.f;
    }
    float ss = 0.f;
#pragma unroll 2
    for (int i = threadIdx.x * V; i < E; i += blockDim.x * V) {
        float x[RT][V], d[V], g[V];
        if (a.start != nullptr) {
            X::load(a.start + t * E + i, x[0]);
#pragma unroll
            for (int e = 0; e < V; ++e) x[0][e] *= a.start_scale;
#pragma unroll
            for (int s = 1; s < RT; ++s)
#pragma unroll
                for (int e = 0; e < V; ++e) x[s][e] = x[0][e];
        } else {
#pragma unroll
            for (int s = 0; s < RT; ++s) {
                if (s < R) X::load(xr + (size_t)s * E + i, x[s]);
                else
#pragma unroll
                    for (int e = 0; e < V; ++e) x[s][e] = 0.f;
            }
        }
        if (has_d) {
            const float *dp = a.d + t * E + i;
            X::load(dp, d);
            if (a.gate != nullptr) X::load(a.gate + t * a.ldg + i, g);
            for (int p0 = 1; p0 < a.n_parts; p0 += 8) {
                float part[8][V];
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    if (p0 + u < a.n_parts) X::load(dp + (size_t)(p0 + u) * a.part_stride, part[u]);
#pragma unroll
                for (int u = 0; u < 8; ++u)
                    if (p0 + u < a.n_parts)
#pragma unroll
                        for (int e = 0; e < V; ++e) d[e] += part[u][e];
            }
            if (a.d_bias != nullptr) {
                float b[V];
                X::load_w(a.d_bias + i, b);
#pragma unroll
                for (int e = 0; e < V; ++e) d[e] += b[e];
            }
            if (a.gate != nullptr)
#pragma unroll
                for (int e = 0; e < V; ++e) d[e] = d[e] / (1.0f + expf(-g[e]));
        }
        float u[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            float y[RT];
            if (has_d) {
#pragma unroll
                for (int q = 0; q < RT; ++q) {
                    y[q] = wout[q] * d[e];
#pragma unroll
                    for (int s = 0; s < RT; ++s) y[q] = fmaf(mix[s][q], x[s][e], y[q]);
                }
#pragma unroll
                for (int q = 0; q < RT; ++q) x[q][e] = y[q];
            }
            u[e] = win[0] * x[0][e];
#pragma unroll
            for (int s = 1; s < RT; ++s) u[e] = fmaf(win[s], x[s][e], u[e]);
            ss = fmaf(u[e], u[e], ss);
        }
        if (write)
#pragma unroll
            for (int s = 0; s < RT; ++s)
                if (s < R) X::store(xr + (size_t)s * E + i, x[s]);
        X::store(us + i, u);
    }
    if (a.w == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)E + a.eps);
    TO *orow = reinterpret_cast<TO *>(a.out) + (size_t)r * E;
    for (int i = threadIdx.x * V; i < E; i += blockDim.x * V) {        // every thread reads back what it wrote itself
        float w[V], y[V];
        X::load_w(a.w + i, w);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = us[i + e] * inv * w[e];
        X::store(orow + i, y);
    }
}
}  // namespace

// x float32 [n, R, E]; start float32 [n, E] or null; d float32 [n_parts][n, E] or null; gate float32 rows of ldg or null;
// w_out [R] and mix [R, R] with d; w_in [R] or null; w [E] or null; rows int32 [n_out] or null (then x is not written); out [n_out, E].
LGML_API int lgml_stream_norm(float *x, const float *start, float start_scale, const float *d, int n_parts, long long part_stride, const float *d_bias,
                              const float *gate, int ldg, const float *w_out, const float *mix, const float *w_in, const float *w, const int *rows,
                              void *out, int out_dtype, int n_out, int E, int R, float eps, cudaStream_t stream) {
    LGML_REQUIRE(n_out >= 0 && E > 0 && R >= 1 && R <= MAX_STREAMS, "stream_norm: rows of %d in %d streams (1 to %d)", E, R, MAX_STREAMS);
    LGML_REQUIRE(d == nullptr || (w_out != nullptr && mix != nullptr && n_parts >= 1), "stream_norm: a result comes with its out and mix weights");
    LGML_REQUIRE(d == nullptr || start == nullptr, "stream_norm: nothing can be pending before the streams start");
    LGML_REQUIRE(start == nullptr || rows == nullptr, "stream_norm: the streams start for all rows");
    LGML_REQUIRE(gate == nullptr || ldg >= E, "stream_norm: the gate's rows are shorter than %d", E);
    LGML_REQUIRE(w == nullptr || out != nullptr, "stream_norm: a norm needs its output");
    LGML_REQUIRE((size_t)E * sizeof(float) <= 200 * 1024, "stream_norm: rows of %d floats do not fit shared memory", E);
    if (n_out == 0) return 0;
    const bool vec = E % 4 == 0 && (gate == nullptr || ldg % 4 == 0) && part_stride % 4 == 0 &&
                     (((uintptr_t)x | (uintptr_t)start | (uintptr_t)d | (uintptr_t)d_bias | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
    StreamArgs a{x, start, start_scale, d, n_parts, part_stride, d_bias, gate, ldg, w_out, mix, w_in, w, rows, out, E, R, eps};
    // few rows (a decode step): a row is latency, so up to 512 threads share it; many rows: blocks of up to 256 fill the SMs
    const int want = vec ? (E + 3) / 4 : E;
    const int most = n_out <= 296 ? 512 : 256;
    int threads = (want + 31) / 32 * 32;
    threads = threads < 32 ? 32 : (threads > most ? most : threads);
    const size_t smem = (size_t)((E + 3) & ~3) * sizeof(float);
#define LGML_ST(TO, RT, V)                                                                                                          \
    do {                                                                                                                            \
        if (smem > 48 * 1024) cudaFuncSetAttribute(stream_norm_kernel<TO, RT, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        lgml_launch(stream_norm_kernel<TO, RT, V>, n_out, threads, smem, stream, a);                                                \
    } while (0)
#define LGML_ST_V(TO, RT) do { if (vec) LGML_ST(TO, RT, 4); else LGML_ST(TO, RT, 1); } while (0)
#define LGML_ST_R(TO) \
    switch (R) { case 1: LGML_ST_V(TO, 1); break; case 2: LGML_ST_V(TO, 2); break; case 3: LGML_ST_V(TO, 3); break; case 4: LGML_ST_V(TO, 4); break; \
                 default: LGML_ST(TO, MAX_STREAMS, 1); }
    if (out_dtype == LGML_F32) { LGML_ST_R(float) }
    else if (out_dtype == LGML_BF16) { LGML_ST_R(__nv_bfloat16) }
    else LGML_FAIL("stream_norm: unknown output type %d", out_dtype);
#undef LGML_ST_R
#undef LGML_ST_V
#undef LGML_ST
    return lgml_launch_status("stream_norm");
}
