// What surrounds the recurrence of a matrix memory with exponential gates (the recurrence itself: ssd_scan with given decays):
//
//   i = cap tanh(z_i / cap),  f = logsigmoid(cap tanh(z_f / cap))               per (token, head), z with its bias added
//   m_t = max(f_t + m_(t-1), i_t)                                               m = 0 when a request starts
//   a_t = exp(f_t + m_(t-1) - m_t),  b_t = exp(i_t - m_t)                       decay and write weight of the recurrence
//   o   = s S_t^T q / (max(s |n_t . q|, exp(-m_t)) + 1e-6)                      s: the factor on q
//   out = o / rms(o) * w * sigmoid(g)                                           per head, w of all heads' size
//
//   memory_gates    a, b and exp(-m) of a step's tokens, request by request; m in the request's state slot
//   memory_output   the last two lines
// All float32; out in the compute type.
#include <math.h>

#include "common.cuh"

LGML_DEFINE_LAST_ERROR(lgml_matrix_memory)

namespace {
constexpr int GATE_THREADS = 512;       // at most; fewer when a step brings few tokens a request

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// Block (request, head).  Every thread takes a run of consecutive tokens: their map m -> max(F + m, I) is composed in order, the
// runs' maps by a scan over the block, and each thread then walks its run from its true start.
// gates [n, 4 H]: a | b | exp(-m) | log a.
__global__ void __launch_bounds__(GATE_THREADS) memory_gates_kernel(const float *__restrict__ zi, const float *__restrict__ zf, int ldz, float cap,
                                                                    float *__restrict__ m_state, long long state_ld, const int *__restrict__ seq_start,
                                                                    const int *__restrict__ slots, float *__restrict__ gates, int H) {
    pdl_trigger();
    pdl_wait();
    __shared__ float Fs[GATE_THREADS], Is[GATE_THREADS], Ms[GATE_THREADS];
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, threads = blockDim.x;
    const int t0 = seq_start[s], n = seq_start[s + 1] - t0;
    if (n <= 0) return;
    float *ms = m_state + (size_t)slots[s] * state_ld + h;
    const float m0 = act_load(ms);
    const int per = (n + threads - 1) / threads;
    const int first = min(tid * per, n), last = min(first + per, n);
    const int ldg = 4 * H;
    float F = 0.f, I = -INFINITY;
#pragma unroll 4
    for (int t = first; t < last; ++t) {
        const float i = capped(act_load(zi + (size_t)(t0 + t) * ldz + h), cap);
        const float f = log_sigmoid(capped(act_load(zf + (size_t)(t0 + t) * ldz + h), cap));
        float *g = gates + (size_t)(t0 + t) * ldg + h;
        g[0] = f, g[H] = i;                     // kept for this thread's second walk
        F += f;
        I = fmaxf(f + I, i);
    }
    Fs[tid] = F, Is[tid] = I;
    __syncthreads();
    for (int o = 1; o < threads && o < n; o <<= 1) {        // inclusive scan: the earlier map first
        float Fp = 0.f, Ip = -INFINITY;
        const bool have = tid >= o;
        if (have) Fp = Fs[tid - o], Ip = Is[tid - o];
        __syncthreads();
        if (have) {
            I = fmaxf(F + Ip, I);
            F = Fp + F;
            Fs[tid] = F, Is[tid] = I;
        }
        __syncthreads();
    }
    float m = tid == 0 ? m0 : fmaxf(Fs[tid - 1] + m0, Is[tid - 1]);
    float m_end = m;
    for (int t = first; t < last; ++t) {
        const float *g = gates + (size_t)(t0 + t) * ldg + h;
        m_end = fmaxf(g[0] + m_end, g[H]);
    }
    Ms[tid] = m_end;
    __syncthreads();
    // the decay of a run's first token is taken from the m that the run before really ended with, so that the decays of a
    // request multiply to what its values of m say, whatever the rounding of the composed maps
    float prev = tid == 0 ? m0 : Ms[tid - 1];
    for (int t = first; t < last; ++t) {
        float *g = gates + (size_t)(t0 + t) * ldg + h;
        const float f = g[0], i = g[H];
        m = fmaxf(f + m, i);
        g[3 * H] = f + prev - m;
        g[0] = expf(f + prev - m);
        g[H] = expf(i - m);
        g[2 * H] = expf(-m);
        prev = m;
    }
    if (first < last && last == n) *ms = m;
}

// y [n, H (P + 1)]: per head S^T q (P numbers), then n . q.  A warp takes a (token, head).
template <typename T>
__global__ void __launch_bounds__(128) memory_output_kernel(const float *__restrict__ y, const float *__restrict__ gates, float q_scale,
                                                            const float *__restrict__ w, const float *__restrict__ gate, int ldg, T *__restrict__ out,
                                                            int ldo, int n_tokens, int H, int P, float eps) {
    pdl_trigger();
    pdl_wait();
    const int lane = threadIdx.x & 31;
    const long long total = (long long)n_tokens * H;
    for (long long u = (long long)blockIdx.x * 4 + (threadIdx.x >> 5); u < total; u += (long long)gridDim.x * 4) {
        const int t = (int)(u / H), h = (int)(u - (long long)t * H);
        const float *row = y + u * (P + 1);
        const float *gr = gate + (size_t)t * ldg + (size_t)h * P, *wr = w + (size_t)h * P;
        T *orow = out + (size_t)t * ldo + (size_t)h * P;
        const float den = fmaxf(fabsf(q_scale * act_load(row + P)), act_load(gates + (size_t)t * 4 * H + 2 * H + h)) + 1e-6f;
        const float k = q_scale / den;
        constexpr int KEEP = 8;                 // entries a lane keeps between the two walks
        float v[KEEP], ss = 0.f;
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const int d = i * 32 + lane;
            v[i] = d < P ? act_load(row + d) * k : 0.f;
            ss = fmaf(v[i], v[i], ss);
        }
        for (int d = KEEP * 32 + lane; d < P; d += 32) {
            const float o = act_load(row + d) * k;
            ss = fmaf(o, o, ss);
        }
        const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)P + eps);
#pragma unroll
        for (int i = 0; i < KEEP; ++i) {
            const int d = i * 32 + lane;
            if (d < P) orow[d] = from_f32<T>(v[i] * inv * __ldg(wr + d) / (1.0f + expf(-act_load(gr + d))));
        }
        for (int d = KEEP * 32 + lane; d < P; d += 32)
            orow[d] = from_f32<T>(act_load(row + d) * k * inv * __ldg(wr + d) / (1.0f + expf(-act_load(gr + d))));
    }
}
}  // namespace

// zi, zf: float32 rows of H entries, ldz apart; m_state: the first slot's m of head 0, slots state_ld apart; gates float32 [n, 4 H].
LGML_API int lgml_memory_gates(const float *zi, const float *zf, int ldz, float cap, float *m_state, long long state_ld, const int *seq_start,
                               const int *slots, float *gates, int n_tokens, int n_seqs, int H, cudaStream_t stream) {
    LGML_REQUIRE(n_seqs >= 0 && H > 0 && H <= 65535 && ldz >= H && cap > 0.f, "memory_gates: bad sizes");
    if (n_seqs == 0) return 0;
    const int threads = n_tokens == n_seqs ? 32 : (n_tokens / n_seqs <= 256 ? 128 : GATE_THREADS);
    lgml_launch(memory_gates_kernel, dim3(n_seqs, H), threads, 0, stream, zi, zf, ldz, cap, m_state, state_ld, seq_start, slots, gates, H);
    return lgml_launch_status("memory_gates");
}

// y float32 [n, H (P + 1)] contiguous; w float32 [H P]; gate: float32 rows, ldg apart; out rows of H P entries, ldo apart.
LGML_API int lgml_memory_output(const float *y, const float *gates, float q_scale, const float *w, const float *gate, int ldg, void *out, int dtype,
                                int ldo, int n_tokens, int H, int P, float eps, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && H > 0 && P > 0 && ldg >= H * P && ldo >= H * P, "memory_output: bad sizes");
    if (n_tokens == 0) return 0;
    const long long blocks = ((long long)n_tokens * H + 3) / 4;
    const int grid = (int)(blocks < 148 * 32 ? blocks : 148 * 32);
    if (dtype == LGML_F32)
        lgml_launch(memory_output_kernel<float>, grid, 128, 0, stream, y, gates, q_scale, w, gate, ldg, (float *)out, ldo, n_tokens, H, P, eps);
    else if (dtype == LGML_BF16)
        lgml_launch(memory_output_kernel<__nv_bfloat16>, grid, 128, 0, stream, y, gates, q_scale, w, gate, ldg, (__nv_bfloat16 *)out, ldo, n_tokens, H, P, eps);
    else
        LGML_FAIL("memory_output: unknown type %d", dtype);
    return lgml_launch_status("memory_output");
}
