// A real-gated linear recurrent unit behind a short convolution, per channel c of request s:
//
//   u_t   = bias_c + sum_j w[j, c] x_(t - taps + 1 + j)              (inputs before the start are zero)
//   r_t   = sigmoid((Ra[b] u_t,b + ra_b)_c),  i_t = sigmoid((Ri[b] u_t,b + ri_b)_c)      b: the part of the channels that holds c
//   a_t   = exp(-8 r_t softplus(lam_c));      S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t
//   out_t = S_t gelu_tanh(y_t)
//
// x | y are the columns of one projection, proj float32 [n, 2 C].  A request's state row, float32: S [C], then a ring of the
// last `taps` inputs, [taps, C], the input of position p in row p mod taps (absent with one tap): what a step of one token
// writes is then not what anyone reads, and every block of channels may work on its own.
//
//   rglru_step    one token a request: convolution, both gates, recurrence and output in one kernel, a block per (8 tokens, 32 channels)
//   rglru_conv    the convolution alone for longer portions; also brings the ring up to date
//   rglru_gates   a_t and the pushed term sqrt(1 - a^2) i u of longer portions as products of 8 rows
//   rglru_finish  the same from logits that a grouped product on tensor cores has left: a group a part of the channels, u in three
//                 bfloat16 pieces side by side (24 bits: what is multiplied is the float32 number)
//   rglru_scan    S_t = a_t S_(t-1) + push_t and the output, a thread a channel of a request
//   rglru_chunks  the same for long portions in three passes: every chunk's (product of a, scan from zero), the chain over
//                 a request's chunks, every chunk again from its true start
//
// Everything here is float32 arithmetic in both compute types (the gates' matrices are in the compute type); only out, which
// feeds a matrix product, is stored in the compute type.
#include <math.h>

#include "common.cuh"
#include "few_rows.cuh"

LGML_DEFINE_LAST_ERROR(lgml_rglru)

namespace {
constexpr int NT = 8;            // tokens a block of the row forms takes
constexpr int CH = 32;           // channels a block of the row forms takes: eight warps of four
constexpr int CHUNK = 32;        // tokens of a chunk of a long portion
constexpr int MAX_TAPS = 16;

// 1 / (1 + e^-v), right to two units in the last place; e^-v is kept below 2^126, where the fast division still divides
__device__ __forceinline__ float sigmoid_(float v) { return __fdividef(1.0f, 1.0f + expf(fminf(-v, 80.0f))); }
__device__ __forceinline__ float gelu_tanh(float z) { return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))); }

// a and the pushed term from the gates' logits; sp8 = 8 softplus(lam)
__device__ __forceinline__ void gate_pair(float zr, float zi, float sp8, float u, float &a, float &push) {
    const float log_a = -sigmoid_(zr) * sp8;
    a = expf(log_a);
    push = sqrtf(-expm1f(2.0f * log_a)) * sigmoid_(zi) * u;
}

// One result of the convolution: the inputs in order, oldest first.  Token t of the step at position pos, its request's first token
// t0; inputs of earlier steps come from the ring.
__device__ __forceinline__ float conv_at(const float *__restrict__ x, int ldx, const float *__restrict__ w, float bias, const float *ring, int C, int taps,
                                         int t, int t0, int pos, int c) {
    float v = bias;
    for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;
        if (pos - back < 0) continue;
        const float in = t - back >= t0 ? act_load(x + (size_t)(t - back) * ldx + c) : act_load(ring + (size_t)((pos - back) % taps) * C + c);
        v = fmaf(__ldg(w + (size_t)j * C + c), in, v);
    }
    return v;
}

// The logits of both gates for the 8 tokens in `us` and the 32 channels from k_out on of part b: zs [2][NT][CH].  A warp takes four
// channels, lane groups of `lanes` a channel at a time.
template <typename T>
__device__ __forceinline__ void gate_logits(const T *__restrict__ ra, const T *__restrict__ ri, const float *us, int ldu, int b, int P, int k_out, int lanes, int vec,
                                            float *zs) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, per = 32 / lanes, sub = lane % lanes;
    for (int j0 = 0; j0 < 4; j0 += per) {
        const int q = j0 + lane / lanes, ch = warp * 4 + q, k = k_out + ch;       // this lane group's channel of the part
        const bool mine = q < 4 && k < P;
        float zr[NT], zi[NT];
#pragma unroll
        for (int j = 0; j < NT; ++j) zr[j] = zi[j] = 0.f;
        if (mine) {
            few_rows_share<T, NT>(ra + ((size_t)b * P + k) * P, us, ldu, P, sub, lanes, vec != 0, zr);
            few_rows_share<T, NT>(ri + ((size_t)b * P + k) * P, us, ldu, P, sub, lanes, vec != 0, zi);
        }
        few_rows_reduce<NT>(zr, lanes);
        few_rows_reduce<NT>(zi, lanes);
        if (mine && sub == 0) {
#pragma unroll
            for (int j = 0; j < NT; ++j) zs[j * CH + ch] = zr[j], zs[(NT + j) * CH + ch] = zi[j];
        }
    }
}

// ---- one token a request ---------------------------------------------------------------------------
// TAPS: the taps at compile time (0: any number).
template <typename T, typename TO, int TAPS>
__global__ void __launch_bounds__(256) rglru_step_kernel(const float *__restrict__ proj, int ldp, const float *__restrict__ conv_w,
                                                         const float *__restrict__ conv_b, float *__restrict__ state, long long state_ld,
                                                         const int *__restrict__ slots, const int *__restrict__ positions, const T *__restrict__ ra,
                                                         const float *__restrict__ ra_b, const T *__restrict__ ri, const float *__restrict__ ri_b,
                                                         const float *__restrict__ sp8, TO *__restrict__ out, int n, int C, int P, int any_taps, int lanes,
                                                         int vec) {
    pdl_trigger();
    // the gates' matrices depend on no earlier kernel: have this block's rows of them in L2 by the time it may go on
    {
        const size_t first = ((size_t)blockIdx.y * P + blockIdx.x * CH) * P, bytes = (size_t)min(CH, P - (int)blockIdx.x * CH) * P * sizeof(T);
        for (size_t o = (size_t)threadIdx.x * 128; o < bytes; o += (size_t)blockDim.x * 128) {
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char *>(ra + first) + o));
            asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char *>(ri + first) + o));
        }
    }
    pdl_wait();
    extern __shared__ __align__(16) float us[];        // u of up to 8 tokens, the whole part of the channels
    __shared__ float zs[2 * NT * CH];
    const int ldu = (P + 3) & ~3, taps = TAPS > 0 ? TAPS : any_taps;
    const int b = blockIdx.y, t0 = blockIdx.z * NT, nt = min(NT, n - t0);
    if (TAPS > 0) {
        // a thread a channel: the inputs of all its tokens are in flight together
        const float *ring[NT];
        int pos[NT];
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const int t = t0 + min(j, nt - 1);
            ring[j] = state + (size_t)slots[t] * state_ld + C, pos[j] = positions[t];
        }
        for (int k = threadIdx.x; k < ldu; k += blockDim.x) {
            const int c = b * P + k;
            float in[NT][TAPS > 0 ? TAPS : 1], w[TAPS > 0 ? TAPS : 1];
#pragma unroll
            for (int j = 0; j < NT; ++j)
#pragma unroll
                for (int i = 0; i < TAPS; ++i) {
                    const int back = TAPS - 1 - i;
                    const bool there = j < nt && k < P && pos[j] >= back;
                    in[j][i] = !there ? 0.f : (back == 0 ? act_load(proj + (size_t)(t0 + j) * ldp + c) : act_load(ring[j] + (size_t)((pos[j] - back) % (TAPS > 0 ? TAPS : 1)) * C + c));
                }
#pragma unroll
            for (int i = 0; i < TAPS; ++i) w[i] = k < P ? __ldg(conv_w + (size_t)i * C + c) : 0.f;
            const float bias = k < P ? __ldg(conv_b + c) : 0.f;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                float v = bias;
#pragma unroll
                for (int i = 0; i < TAPS; ++i) v = fmaf(w[i], in[j][i], v);
                us[j * ldu + k] = j < nt ? v : 0.f;
            }
        }
    } else {
        for (int e = threadIdx.x; e < NT * ldu; e += blockDim.x) {
            const int j = e / ldu, k = e - j * ldu;
            float u = 0.f;
            if (j < nt && k < P) {
                const int t = t0 + j, c = b * P + k;
                u = conv_at(proj, ldp, conv_w, conv_b[c], state + (size_t)slots[t] * state_ld + C, C, taps, t, t, positions[t], c);
            }
            us[e] = u;
        }
    }
    // a thread finishes one channel of one token: what it needs beside the logits is on its way meanwhile
    const int my_j = threadIdx.x / CH, my_k = blockIdx.x * CH + threadIdx.x % CH;
    const bool mine = my_j < nt && my_k < P;
    const int t = t0 + my_j, c = b * P + my_k;
    float *row = nullptr;
    float s_old = 0.f, y = 0.f, x_in = 0.f;
    int pos_t = 0;
    if (mine) {
        row = state + (size_t)slots[t] * state_ld, pos_t = positions[t];
        s_old = act_load(row + c), y = act_load(proj + (size_t)t * ldp + C + c), x_in = act_load(proj + (size_t)t * ldp + c);
    }
    __syncthreads();
    gate_logits<T>(ra, ri, us, ldu, b, P, blockIdx.x * CH, lanes, vec, zs);
    __syncthreads();
    if (!mine) return;
    float a, push;
    gate_pair(zs[my_j * CH + threadIdx.x % CH] + ra_b[c], zs[(NT + my_j) * CH + threadIdx.x % CH] + ri_b[c], sp8[c], us[my_j * ldu + my_k], a, push);
    const float S = fmaf(a, s_old, push);
    row[c] = S;
    out[(size_t)t * C + c] = from_f32<TO>(S * gelu_tanh(y));
    if (taps > 1) row[C + (size_t)(pos_t % taps) * C + c] = x_in;
}

// A convolved input on its way out: a float32 number at [t, c], or three bfloat16 numbers whose sum it is (8 + 8 + 8 bits): channel
// k of part b of token t in row b * rows + t of a matrix [B rows, 3 P], at columns k, P + k and 2 P + k.  A product of such rows with [R | R | R] is
// R times the float32 number.
struct AsFloat {
    float *u;
    int C;
    __device__ __forceinline__ void put(int t, int c, float v) const { u[(size_t)t * C + c] = v; }
    __device__ __forceinline__ void put4(int t, int c, const float4 &v) const { *reinterpret_cast<float4 *>(u + (size_t)t * C + c) = v; }
};
struct AsPieces {
    __nv_bfloat16 *u;
    int rows, P;
    __device__ __forceinline__ __nv_bfloat16 *at(int t, int c) const {
        const int b = c / P;
        return u + ((size_t)b * rows + t) * 3 * P + (c - b * P);
    }
    __device__ __forceinline__ void put(int t, int c, float v) const {
        __nv_bfloat16 *p = at(t, c);
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            const __nv_bfloat16 h = __float2bfloat16_rn(v);
            p[k * P] = h;
            v -= __bfloat162float(h);
        }
    }
    __device__ __forceinline__ void put4(int t, int c, const float4 &v) const {       // parts are multiples of 8 channels
        __nv_bfloat16 *p = at(t, c);
        float x[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int k = 0; k < 3; ++k) {
            __nv_bfloat162 lo = __floats2bfloat162_rn(x[0], x[1]), hi = __floats2bfloat162_rn(x[2], x[3]);
            *reinterpret_cast<uint2 *>(p + k * P) = make_uint2(*reinterpret_cast<unsigned *>(&lo), *reinterpret_cast<unsigned *>(&hi));
            x[0] -= __low2float(lo), x[1] -= __high2float(lo), x[2] -= __low2float(hi), x[3] -= __high2float(hi);
        }
    }
    // two neighbouring channels (c even) in three 4-byte loads
    __device__ __forceinline__ float2 get2(int t, int c) const {
        const unsigned *p = reinterpret_cast<const unsigned *>(at(t, c));
        const unsigned hi = act_load(p), mid = act_load(p + P / 2), lo = act_load(p + P);
        auto first = [](unsigned w) { return __uint_as_float(w << 16); };
        auto second = [](unsigned w) { return __uint_as_float(w & 0xffff0000u); };
        return make_float2(first(hi) + (first(mid) + first(lo)), second(hi) + (second(mid) + second(lo)));
    }
};

// ---- the convolution of longer portions ----------------------------------------------------------------
// A thread takes one channel of one token.  The thread of a request's first token computes every token that reaches into
// the ring and then writes the step's last taps - 1 inputs there; nobody else touches those floats.
template <typename OUT>
__global__ void __launch_bounds__(256) rglru_conv_kernel(const float *__restrict__ proj, int ldp, const float *__restrict__ conv_w,
                                                         const float *__restrict__ conv_b, float *__restrict__ state, long long state_ld,
                                                         const int *__restrict__ seq_of_token, const int *__restrict__ seq_start,
                                                         const int *__restrict__ slots, const int *__restrict__ positions, const OUT u, int n, int C,
                                                         int taps) {
    pdl_trigger();
    pdl_wait();
    const size_t total = (size_t)n * C;
    for (size_t it = (size_t)blockIdx.x * blockDim.x + threadIdx.x; it < total; it += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(it / C), c = (int)(it - (size_t)t * C);
        const int s = seq_of_token[t], t0 = seq_start[s];
        const float bias = __ldg(conv_b + c);
        if (t == t0) {
            float *ring = state + (size_t)slots[s] * state_ld + C;
            const int t1 = seq_start[s + 1], last = min(t1, t0 + max(taps - 1, 1)), pos0 = positions[t0];
            for (int i = t0; i < last; ++i) u.put(i, c, conv_at(proj, ldp, conv_w, bias, ring, C, taps, i, t0, pos0 + i - t0, c));
            if (taps > 1)
                for (int i = max(t0, t1 - (taps - 1)); i < t1; ++i) ring[(size_t)((pos0 + i - t0) % taps) * C + c] = act_load(proj + (size_t)i * ldp + c);
        } else if (t - t0 >= taps - 1) {
            u.put(t, c, conv_at(proj, ldp, conv_w, bias, nullptr, C, taps, t, t0, positions[t], c));
        }
    }
}

// The same for many tokens, four channels a thread and four tokens in a row (a row of inputs is read once for four results): tokens
// 4 i .. 4 i + 3 of the step, whichever requests they belong to.  Taps at compile time, C a multiple of 4.
template <int TAPS, typename OUT>
__global__ void __launch_bounds__(256) rglru_conv_runs_kernel(const float *__restrict__ proj, int ldp, const float *__restrict__ conv_w,
                                                              const float *__restrict__ conv_b, float *__restrict__ state, long long state_ld,
                                                              const int *__restrict__ seq_of_token, const int *__restrict__ seq_start,
                                                              const int *__restrict__ slots, const int *__restrict__ positions, const OUT u, int n,
                                                              int C) {
    pdl_trigger();
    pdl_wait();
    constexpr int RUN = 4;
    const int quads = C / 4;
    const size_t total = (size_t)((n + RUN - 1) / RUN) * quads;
    for (size_t it = (size_t)blockIdx.x * blockDim.x + threadIdx.x; it < total; it += (size_t)gridDim.x * blockDim.x) {
        const int ta = (int)(it / quads) * RUN, c = (int)(it - (size_t)(ta / RUN) * quads) * 4, tb = min(n, ta + RUN);
        float4 w[TAPS];
#pragma unroll
        for (int j = 0; j < TAPS; ++j) w[j] = __ldg(reinterpret_cast<const float4 *>(conv_w + (size_t)j * C + c));
        const float4 bias = __ldg(reinterpret_cast<const float4 *>(conv_b + c));
        float4 in[RUN + TAPS - 1];
#pragma unroll
        for (int k = 0; k < RUN + TAPS - 1; ++k) {
            const int t = ta - (TAPS - 1) + k;
            in[k] = t >= 0 && t < tb ? act_load(reinterpret_cast<const float4 *>(proj + (size_t)t * ldp + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < RUN; ++i) {
            const int t = ta + i;
            if (t >= tb) break;
            const int s = seq_of_token[t], t0 = seq_start[s];
            if (t - t0 >= TAPS - 1) {
                float4 v = bias;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    v.x = fmaf(w[j].x, in[i + j].x, v.x), v.y = fmaf(w[j].y, in[i + j].y, v.y);
                    v.z = fmaf(w[j].z, in[i + j].z, v.z), v.w = fmaf(w[j].w, in[i + j].w, v.w);
                }
                u.put4(t, c, v);
            } else if (t == t0) {
                float *ring = state + (size_t)slots[s] * state_ld + C;
                const int t1 = seq_start[s + 1], last = min(t1, t0 + max(TAPS - 1, 1)), pos0 = positions[t0];
                for (int e = 0; e < 4; ++e) {
                    for (int k = t0; k < last; ++k)
                        u.put(k, c + e, conv_at(proj, ldp, conv_w, __ldg(conv_b + c + e), ring, C, TAPS, k, t0, pos0 + k - t0, c + e));
                    if (TAPS > 1)
                        for (int k = max(t0, t1 - (TAPS - 1)); k < t1; ++k)
                            ring[(size_t)((pos0 + k - t0) % TAPS) * C + c + e] = act_load(proj + (size_t)k * ldp + c + e);
                }
            }
        }
    }
}

// ---- the gates of longer portions -------------------------------------------------------------------------
// u float32 [n, C] -> ab float32 [2, n, C]: a, then the pushed term
template <typename T>
__global__ void __launch_bounds__(256) rglru_gates_rows_kernel(const float *__restrict__ u, const T *__restrict__ ra, const float *__restrict__ ra_b,
                                                               const T *__restrict__ ri, const float *__restrict__ ri_b, const float *__restrict__ sp8,
                                                               float *__restrict__ ab, int n, int C, int P, int lanes, int vec) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float us[];
    __shared__ float zs[2 * NT * CH];
    const int ldu = (P + 3) & ~3;
    const int b = blockIdx.y, t0 = blockIdx.x * NT, nt = min(NT, n - t0);
    for (int e = threadIdx.x; e < NT * ldu; e += blockDim.x) {
        const int j = e / ldu, k = e - j * ldu;
        us[e] = j < nt && k < P ? act_load(u + (size_t)(t0 + j) * C + b * P + k) : 0.f;
    }
    __syncthreads();
    gate_logits<T>(ra, ri, us, ldu, b, P, blockIdx.z * CH, lanes, vec, zs);
    __syncthreads();
    const int j = threadIdx.x / CH, ch = threadIdx.x % CH, k = blockIdx.z * CH + ch, c = b * P + k;
    if (j >= nt || k >= P) return;
    float a, push;
    gate_pair(zs[j * CH + ch] + ra_b[c], zs[(NT + j) * CH + ch] + ri_b[c], sp8[c], us[j * ldu + k], a, push);
    ab[(size_t)(t0 + j) * C + c] = a;
    ab[(size_t)(n + t0 + j) * C + c] = push;
}

// Many tokens in bfloat16: the gates' logits come from a product on tensor cores over the inputs in pieces, z float32 [B rows, 2 P]: row b *
// rows + t, the decay gate's at column k, the input gate's at P + k.  A thread takes two neighbouring channels of a token, or, with chunks, of a
// chunk's tokens, and then also forms the chunk's product of a and its scan from zero (pass 1 of the recurrence below).
struct GatePair {
    float2 zr, zi, u;
    __device__ __forceinline__ void load(const float *__restrict__ z, const AsPieces &in, int t, int c, int b, int k) {
        const float *row = z + ((size_t)b * in.rows + t) * 2 * in.P + k;
        zr = act_load(reinterpret_cast<const float2 *>(row)), zi = act_load(reinterpret_cast<const float2 *>(row + in.P));
        u = in.get2(t, c);
    }
    __device__ __forceinline__ void finish(const float2 &br, const float2 &bi, const float2 &sp, float2 &a, float2 &push) const {
        gate_pair(zr.x + br.x, zi.x + bi.x, sp.x, u.x, a.x, push.x);
        gate_pair(zr.y + br.y, zi.y + bi.y, sp.y, u.y, a.y, push.y);
    }
};
__global__ void __launch_bounds__(256) rglru_finish_kernel(const float *__restrict__ z, const AsPieces u, const float *__restrict__ ra_b,
                                                           const float *__restrict__ ri_b, const float *__restrict__ sp8, float *__restrict__ ab, int n, int C) {
    pdl_trigger();
    pdl_wait();
    const size_t total = (size_t)n * (C / 2);
    for (size_t it = (size_t)blockIdx.x * blockDim.x + threadIdx.x; it < total; it += (size_t)gridDim.x * blockDim.x) {
        const int t = (int)(it / (C / 2)), c = (int)(it - (size_t)t * (C / 2)) * 2, b = c / u.P;
        GatePair g;
        g.load(z, u, t, c, b, c - b * u.P);
        float2 a, push;
        g.finish(__ldg(reinterpret_cast<const float2 *>(ra_b + c)), __ldg(reinterpret_cast<const float2 *>(ri_b + c)), __ldg(reinterpret_cast<const float2 *>(sp8 + c)),
                 a, push);
        *reinterpret_cast<float2 *>(ab + (size_t)t * C + c) = a;
        *reinterpret_cast<float2 *>(ab + ((size_t)n + t) * C + c) = push;
    }
}
__global__ void __launch_bounds__(64, 14) rglru_finish_chunks_kernel(const float *__restrict__ z, const AsPieces u, const float *__restrict__ ra_b,
                                                                 const float *__restrict__ ri_b, const float *__restrict__ sp8, float *__restrict__ ab,
                                                                 const int *__restrict__ chunks, float *__restrict__ A, float *__restrict__ B, int n, int C) {
    pdl_trigger();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 2, k = blockIdx.y;
    if (c >= C) return;
    const int b = c / u.P;
    const float2 br = __ldg(reinterpret_cast<const float2 *>(ra_b + c)), bi = __ldg(reinterpret_cast<const float2 *>(ri_b + c));
    const float2 sp = __ldg(reinterpret_cast<const float2 *>(sp8 + c));
    pdl_wait();
    const int t0 = chunks[2 * k], t1 = chunks[2 * k + 1];
    float2 prod = make_float2(1.f, 1.f), S = make_float2(0.f, 0.f);
    constexpr int W = 8;            // tokens whose loads are in flight together
    for (int t = t0; t < t1; t += W) {
        GatePair g[W];
#pragma unroll
        for (int i = 0; i < W; ++i)
            if (t + i < t1) g[i].load(z, u, t + i, c, b, c - b * u.P);
#pragma unroll
        for (int i = 0; i < W; ++i)
            if (t + i < t1) {
                float2 a, p;
                g[i].finish(br, bi, sp, a, p);
                *reinterpret_cast<float2 *>(ab + (size_t)(t + i) * C + c) = a;
                *reinterpret_cast<float2 *>(ab + ((size_t)n + t + i) * C + c) = p;
                S.x = fmaf(a.x, S.x, p.x), S.y = fmaf(a.y, S.y, p.y);
                prod.x *= a.x, prod.y *= a.y;
            }
    }
    *reinterpret_cast<float2 *>(A + (size_t)k * C + c) = prod;
    *reinterpret_cast<float2 *>(B + (size_t)k * C + c) = S;
}

// ---- the recurrence ---------------------------------------------------------------------------------------
// ab float32 [2, n, C]; y: columns C .. 2 C - 1 of proj.  A thread owns one channel of one request (or of one chunk, from S0) and walks
// its tokens in order; the loads of AHEAD tokens are in flight at a time.
constexpr int AHEAD = 8;
template <typename TO>
__device__ __forceinline__ float walk(const float *__restrict__ ab, const float *__restrict__ proj, int ldp, TO *__restrict__ out, int n, int C, int c, int t0,
                                      int t1, float S) {
    for (int t = t0; t < t1; t += AHEAD) {
        float a[AHEAD], b[AHEAD], y[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (t + i < t1) {
                a[i] = act_load(ab + (size_t)(t + i) * C + c), b[i] = act_load(ab + (size_t)(n + t + i) * C + c);
                y[i] = act_load(proj + (size_t)(t + i) * ldp + C + c);
            }
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (t + i < t1) {
                S = fmaf(a[i], S, b[i]);
                out[(size_t)(t + i) * C + c] = from_f32<TO>(S * gelu_tanh(y[i]));
            }
    }
    return S;
}

template <typename TO>
__global__ void __launch_bounds__(128) rglru_scan_kernel(const float *__restrict__ ab, const float *__restrict__ proj, int ldp, float *__restrict__ state,
                                                         long long state_ld, const int *__restrict__ seq_start, const int *__restrict__ slots,
                                                         TO *__restrict__ out, int n, int C) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    if (c >= C) return;
    float *st = state + (size_t)slots[s] * state_ld + c;
    *st = walk<TO>(ab, proj, ldp, out, n, C, c, seq_start[s], seq_start[s + 1], act_load(st));
}

// pass 1: per (chunk, channel): A = prod a, B = the scan's end from S = 0
__global__ void __launch_bounds__(128) rglru_chunk_ends_kernel(const float *__restrict__ ab, const int *__restrict__ chunks, float *__restrict__ A,
                                                               float *__restrict__ B, int n, int C) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, k = blockIdx.y;
    if (c >= C) return;
    const int t0 = chunks[2 * k], t1 = chunks[2 * k + 1];
    float prod = 1.f, S = 0.f;
    for (int t = t0; t < t1; t += AHEAD) {
        float a[AHEAD], b[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (t + i < t1) a[i] = act_load(ab + (size_t)(t + i) * C + c), b[i] = act_load(ab + (size_t)(n + t + i) * C + c);
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (t + i < t1) S = fmaf(a[i], S, b[i]), prod *= a[i];
    }
    A[(size_t)k * C + c] = prod, B[(size_t)k * C + c] = S;
}

// pass 2: per (request, channel): S at the start of every chunk (written over B), and the slot's new state
__global__ void __launch_bounds__(128) rglru_chain_kernel(const float *__restrict__ A, float *__restrict__ B, const int *__restrict__ chunk_start,
                                                          float *__restrict__ state, long long state_ld, const int *__restrict__ slots, int C) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, s = blockIdx.y;
    if (c >= C) return;
    float *st = state + (size_t)slots[s] * state_ld + c;
    float S = act_load(st);
    const int k1 = chunk_start[s + 1];
    for (int k = chunk_start[s]; k < k1; k += AHEAD) {
        float a[AHEAD], b[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (k + i < k1) a[i] = act_load(A + (size_t)(k + i) * C + c), b[i] = act_load(B + (size_t)(k + i) * C + c);
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (k + i < k1) {
                B[(size_t)(k + i) * C + c] = S;
                S = fmaf(a[i], S, b[i]);
            }
    }
    *st = S;
}

// pass 3: every chunk from its true start
template <typename TO>
__global__ void __launch_bounds__(128) rglru_chunk_scan_kernel(const float *__restrict__ ab, const float *__restrict__ proj, int ldp,
                                                               const int *__restrict__ chunks, const float *__restrict__ S0, TO *__restrict__ out, int n, int C) {
    pdl_trigger();
    pdl_wait();
    const int c = blockIdx.x * blockDim.x + threadIdx.x, k = blockIdx.y;
    if (c >= C) return;
    walk<TO>(ab, proj, ldp, out, n, C, c, chunks[2 * k], chunks[2 * k + 1], act_load(S0 + (size_t)k * C + c));
}
}  // namespace

LGML_API int lgml_rglru_chunk_tokens(void) { return CHUNK; }

#define RGLRU_SIZES(who)                                                                                                                       \
    LGML_REQUIRE(n_tokens >= 0 && C > 0 && P > 0 && C % P == 0 && C / P <= 65535, who ": %d channels in parts of %d", C, P);                   \
    LGML_REQUIRE(dtype == LGML_F32 || dtype == LGML_BF16, who ": unknown type %d", dtype)

// One token a request, n_tokens of them.  ra, ri: [C / P, P, P] in `dtype`; ra_b, ri_b, sp8 (8 softplus(lam)), conv_b float32 [C]; conv_w float32 [taps, C];
// state rows: C floats, then the ring.
LGML_API int lgml_rglru_step(const float *proj, int ldp, const float *conv_w, const float *conv_b, float *state, long long state_ld, const int *slots,
                             const int *positions, const void *ra, const float *ra_b, const void *ri, const float *ri_b, const float *sp8, void *out, int dtype,
                             int n_tokens, int C, int P, int taps, cudaStream_t stream) {
    RGLRU_SIZES("rglru_step");
    LGML_REQUIRE(taps >= 1 && taps <= MAX_TAPS && ldp >= 2 * C && state_ld >= C + (taps > 1 ? (long long)taps * C : 0), "rglru_step: bad strides or taps");
    const size_t smem = sizeof(float) * NT * (size_t)((P + 3) & ~3);
    LGML_REQUIRE(smem <= 48 * 1024, "rglru_step: parts of %d channels are too wide", P);
    LGML_REQUIRE((n_tokens + NT - 1) / NT <= 65535, "rglru_step: too many tokens");
    if (n_tokens == 0) return 0;
    dim3 grid((P + CH - 1) / CH, C / P, (n_tokens + NT - 1) / NT);
#define RGLRU_STEP(T, TAPS)                                                                                                                        \
    lgml_launch(rglru_step_kernel<T, T, TAPS>, grid, 256, smem, stream, proj, ldp, conv_w, conv_b, state, state_ld, slots, positions, (const T *)ra, \
                ra_b, (const T *)ri, ri_b, sp8, (T *)out, n_tokens, C, P, taps, few_rows_lanes<T>(P), few_rows_vec<T>(ra, P) && few_rows_vec<T>(ri, P) ? 1 : 0)
#define RGLRU_STEP_TAPS(T)                 \
    switch (taps) {                        \
        case 2: RGLRU_STEP(T, 2); break;   \
        case 3: RGLRU_STEP(T, 3); break;   \
        case 4: RGLRU_STEP(T, 4); break;   \
        default: RGLRU_STEP(T, 0);         \
    }
    if (dtype == LGML_F32) { RGLRU_STEP_TAPS(float) } else { RGLRU_STEP_TAPS(__nv_bfloat16) }
#undef RGLRU_STEP_TAPS
#undef RGLRU_STEP
    return lgml_launch_status("rglru_step");
}

template <typename OUT>
static int conv_run(const float *proj, int ldp, const float *conv_w, const float *conv_b, float *state, long long state_ld, const int *seq_of_token,
                    const int *seq_start, const int *slots, const int *positions, const OUT &u, bool vec, int n_tokens, int C, int taps, cudaStream_t stream) {
    if (vec && n_tokens >= 64 && taps >= 2 && taps <= 4) {
        const size_t items = (size_t)((n_tokens + 3) / 4) * (C / 4);
        const int blocks = (int)((items + 255) / 256 < 148 * 16 ? (items + 255) / 256 : 148 * 16);
#define RGLRU_RUNS(TT) \
    lgml_launch(rglru_conv_runs_kernel<TT, OUT>, blocks, 256, 0, stream, proj, ldp, conv_w, conv_b, state, state_ld, seq_of_token, seq_start, slots, positions, u, n_tokens, C)
        if (taps == 2) RGLRU_RUNS(2);
        else if (taps == 3) RGLRU_RUNS(3);
        else RGLRU_RUNS(4);
#undef RGLRU_RUNS
        return lgml_launch_status("rglru_conv");
    }
    const size_t items = (size_t)n_tokens * C;
    const int blocks = (int)((items + 255) / 256 < 148 * 16 ? (items + 255) / 256 : 148 * 16);
    lgml_launch(rglru_conv_kernel<OUT>, blocks, 256, 0, stream, proj, ldp, conv_w, conv_b, state, state_ld, seq_of_token, seq_start, slots, positions, u, n_tokens,
                C, taps);
    return lgml_launch_status("rglru_conv");
}

// u: float32 [n, C], or (part > 0) bfloat16 [C / part * rows, 3 part], three numbers whose sum is the float32 one (AsPieces)
LGML_API int lgml_rglru_conv(const float *proj, int ldp, const float *conv_w, const float *conv_b, float *state, long long state_ld, const int *seq_of_token,
                             const int *seq_start, const int *slots, const int *positions, void *u, int part, int rows, int n_tokens, int C, int taps, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && C > 0 && taps >= 1 && taps <= MAX_TAPS && ldp >= C && state_ld >= C + (taps > 1 ? (long long)taps * C : 0), "rglru_conv: bad sizes");
    if (n_tokens == 0) return 0;
    const bool vec = C % 4 == 0 && ldp % 4 == 0 && (((uintptr_t)proj | (uintptr_t)conv_w | (uintptr_t)conv_b | (uintptr_t)u) & 15) == 0;
    if (part) {
        LGML_REQUIRE(part > 0 && part % 8 == 0 && C % part == 0 && rows >= n_tokens, "rglru_conv: pieces of parts of %d channels, %d rows a part", part, rows);
        return conv_run(proj, ldp, conv_w, conv_b, state, state_ld, seq_of_token, seq_start, slots, positions, AsPieces{(__nv_bfloat16 *)u, rows, part}, vec, n_tokens,
                        C, taps, stream);
    }
    return conv_run(proj, ldp, conv_w, conv_b, state, state_ld, seq_of_token, seq_start, slots, positions, AsFloat{(float *)u, C}, vec, n_tokens, C, taps, stream);
}

// The gates as products of 8 rows: u float32 [n, C] -> ab float32 [2, n, C].
LGML_API int lgml_rglru_gates(const float *u, const void *ra, const float *ra_b, const void *ri, const float *ri_b, const float *sp8, float *ab,
                              int dtype, int n_tokens, int C, int P, cudaStream_t stream) {
    RGLRU_SIZES("rglru_gates");
    if (n_tokens == 0) return 0;
    const size_t smem = sizeof(float) * NT * (size_t)((P + 3) & ~3);
    LGML_REQUIRE(smem <= 48 * 1024, "rglru_gates: parts of %d channels are too wide", P);
    dim3 grid((n_tokens + NT - 1) / NT, C / P, (P + CH - 1) / CH);
    if (dtype == LGML_F32)
        lgml_launch(rglru_gates_rows_kernel<float>, grid, 256, smem, stream, u, (const float *)ra, ra_b, (const float *)ri, ri_b, sp8, ab, n_tokens, C, P,
                    few_rows_lanes<float>(P), few_rows_vec<float>(ra, P) && few_rows_vec<float>(ri, P) ? 1 : 0);
    else
        lgml_launch(rglru_gates_rows_kernel<__nv_bfloat16>, grid, 256, smem, stream, u, (const __nv_bfloat16 *)ra, ra_b, (const __nv_bfloat16 *)ri, ri_b, sp8, ab,
                    n_tokens, C, P, few_rows_lanes<__nv_bfloat16>(P), few_rows_vec<__nv_bfloat16>(ra, P) && few_rows_vec<__nv_bfloat16>(ri, P) ? 1 : 0);
    return lgml_launch_status("rglru_gates");
}

// The gates from their logits: z float32 [C / P * rows, 2 P] over the inputs in pieces u bfloat16 [C / P * rows, 3 P].  With chunks (int32 [n_chunks, 2]) also
// every chunk's product of a and scan from zero, scratch float32 [2, n_chunks, C].
LGML_API int lgml_rglru_finish(const float *z, const void *u, int rows, const float *ra_b, const float *ri_b, const float *sp8, float *ab, const int *chunks,
                               int n_chunks, float *scratch, int n_tokens, int C, int P, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && C > 0 && P > 0 && C % P == 0 && P % 8 == 0 && rows >= n_tokens && n_chunks >= 0 && n_chunks <= 65535, "rglru_finish: bad sizes");
    LGML_REQUIRE((((uintptr_t)z | (uintptr_t)u | (uintptr_t)ra_b | (uintptr_t)ri_b | (uintptr_t)sp8 | (uintptr_t)ab | (uintptr_t)scratch) & 15) == 0,
                 "rglru_finish: operands must be 16-byte aligned");
    if (n_tokens == 0) return 0;
    const AsPieces in{(__nv_bfloat16 *)u, rows, P};
    if (chunks != nullptr) {
        lgml_launch(rglru_finish_chunks_kernel, dim3((C / 2 + 63) / 64, n_chunks), 64, 0, stream, z, in, ra_b, ri_b, sp8, ab, chunks, scratch,
                    scratch + (size_t)n_chunks * C, n_tokens, C);
    } else {
        const size_t items = ((size_t)n_tokens * (C / 2) + 255) / 256;
        lgml_launch(rglru_finish_kernel, (int)(items < 148 * 16 ? items : 148 * 16), 256, 0, stream, z, in, ra_b, ri_b, sp8, ab, n_tokens, C);
    }
    return lgml_launch_status("rglru_finish");
}

LGML_API int lgml_rglru_scan(const float *ab, const float *proj, int ldp, float *state, long long state_ld, const int *seq_start, const int *slots, void *out,
                             int dtype, int n_tokens, int n_seqs, int C, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && n_seqs >= 0 && n_seqs <= 65535 && C > 0 && ldp >= 2 * C && state_ld >= C, "rglru_scan: bad sizes");
    if (n_tokens == 0 || n_seqs == 0) return 0;
    dim3 grid((C + 127) / 128, n_seqs);
    if (dtype == LGML_F32)
        lgml_launch(rglru_scan_kernel<float>, grid, 128, 0, stream, ab, proj, ldp, state, state_ld, seq_start, slots, (float *)out, n_tokens, C);
    else if (dtype == LGML_BF16)
        lgml_launch(rglru_scan_kernel<__nv_bfloat16>, grid, 128, 0, stream, ab, proj, ldp, state, state_ld, seq_start, slots, (__nv_bfloat16 *)out, n_tokens, C);
    else
        LGML_FAIL("rglru_scan: unknown type %d", dtype);
    return lgml_launch_status("rglru_scan");
}

// chunks int32 [n_chunks, 2]: token rows [first, past the last), a request's chunks in a row; chunk_start int32 [n_seqs + 1]; scratch float32 [2, n_chunks, C],
// with ends_known = 1 already holding pass 1's results (lgml_rglru_finish)
LGML_API int lgml_rglru_chunks(const float *ab, const float *proj, int ldp, float *state, long long state_ld, const int *chunks, const int *chunk_start,
                               int n_chunks, const int *slots, float *scratch, int ends_known, void *out, int dtype, int n_tokens, int n_seqs, int C,
                               cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && n_chunks >= 0 && n_chunks <= 65535 && n_seqs >= 0 && n_seqs <= 65535 && C > 0 && ldp >= 2 * C && state_ld >= C, "rglru_chunks: bad sizes");
    if (n_chunks == 0) return 0;
    float *A = scratch, *B = scratch + (size_t)n_chunks * C;
    dim3 grid((C + 127) / 128, n_chunks), chain((C + 127) / 128, n_seqs);
    if (!ends_known) lgml_launch(rglru_chunk_ends_kernel, grid, 128, 0, stream, ab, chunks, A, B, n_tokens, C);
    lgml_launch(rglru_chain_kernel, chain, 128, 0, stream, (const float *)A, B, chunk_start, state, state_ld, slots, C);
    if (dtype == LGML_F32)
        lgml_launch(rglru_chunk_scan_kernel<float>, grid, 128, 0, stream, ab, proj, ldp, chunks, (const float *)B, (float *)out, n_tokens, C);
    else if (dtype == LGML_BF16)
        lgml_launch(rglru_chunk_scan_kernel<__nv_bfloat16>, grid, 128, 0, stream, ab, proj, ldp, chunks, (const float *)B, (__nv_bfloat16 *)out, n_tokens, C);
    else
        LGML_FAIL("rglru_chunks: unknown type %d", dtype);
    return lgml_launch_status("rglru_chunks");
}
