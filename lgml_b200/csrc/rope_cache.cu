// Rotary position encoding of q and k, and the write of k and v into the paged cache, in
// one pass over the projection's output.  q is rotated (in place, or into its own buffer);
// k is rotated and stored; v is stored (lua/lgml/transformer.lua:1775, :1788 for the
// rotation; :1838-1839 and :2405-2406 for set_rows into the pool; cell of position p =
// table[p / page] * page + p % page, :1126-1133).  Angles are formed in float32 arithmetic
// without losing what a single float32 product would (rope_sincos).  The input may also be the float32 partial sums of a projection that was cut
// along K: they are added in order (and the bias after them) as they are read.
#include "common.cuh"

LGML_DEFINE_LAST_ERROR(lgml_rope_cache)

namespace {
constexpr int ITEMS = 256;   // work items (pairs of elements) per block

// One work item = one pair of elements of one head of one token.
//   heads 0 .. H-1: q, rotated, written to q_out;   H .. H+Hkv-1: k, rotated, to the cache;
//   H+Hkv .. H+2Hkv-1: v, copied to the cache.
// pairing 0: pairs (i, i + n_rot/2) ("half", the order safetensors checkpoints hold);
// pairing 1: pairs (2i, 2i+1) ("adjacent", the reference's "normal" mode on gguf rows).
// Dimensions at and past n_rot are paired (2j, 2j+1) and pass through unrotated.
template <typename TS, typename T>
__global__ void __launch_bounds__(ITEMS) rope_kv_write_kernel(
    const TS *__restrict__ src, int lds, int n_parts, long long part_stride, const float *__restrict__ bias,
    T *__restrict__ q_out, int ldq, const int *__restrict__ positions, const int *__restrict__ seq_of_token,
    const int *__restrict__ block_table, int max_blocks, const float *__restrict__ inv_freq, const float *__restrict__ inv_freq_lo, int n_rot, int pairing,
    T *__restrict__ k_pages, T *__restrict__ v_pages, int n_pages, int page_size, int H, int Hkv, int D, int write_kv,
    int *__restrict__ status) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const int half_d = D / 2;
    const int n_heads = write_kv ? H + 2 * Hkv : H;
    const int item = blockIdx.y * ITEMS + threadIdx.x;
    if (item >= n_heads * half_d) return;
    const int head = item / half_d, j = item - head * half_d;
    const int pos = positions[t];
    const int half_rot = n_rot / 2;

    // which two dimensions, and whether they turn
    int d0, d1, fi = -1;
    if (head < H + Hkv && j < half_rot) {
        fi = j;
        d0 = pairing ? 2 * j : j;
        d1 = pairing ? 2 * j + 1 : j + half_rot;
    } else if (head < H + Hkv) {
        d0 = n_rot + 2 * (j - half_rot);
        d1 = d0 + 1;
    } else {
        d0 = 2 * j;
        d1 = d0 + 1;
    }
    const size_t col = (size_t)head * D;
    const TS *row = src + (size_t)t * lds + col;
    // Every load goes out before anything waits for one: the elements and their other parts, the
    // bias, the frequency, and the chain position -> block -> page for the cell of the cache (two
    // trips to L2 one after the other, which used to begin only when the rotation was done).
    float a = to_f32(act_load(row + d0)), b = to_f32(act_load(row + d1));
    const float bias0 = bias ? bias[col + d0] : 0.f, bias1 = bias ? bias[col + d1] : 0.f;
    const float f = fi >= 0 ? inv_freq[fi] : 0.f, f_lo = (fi >= 0 && inv_freq_lo) ? inv_freq_lo[fi] : 0.f;
    int page = -1;      // where this token's k and v go
    if (head >= H) {
        const int seq = seq_of_token[t];
        const int blk = pos / page_size;
        if (pos >= 0 && blk < max_blocks) page = block_table[(size_t)seq * max_blocks + blk];
    }
    // the other parts in order; the loads of up to eight of them are issued before the first is used
    // (one after the other they would cost a round trip to L2 each)
    for (int p0 = 1; p0 < n_parts; p0 += 8) {
        float ea[8], eb[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (p0 + u < n_parts) {
                ea[u] = to_f32(act_load(row + (size_t)(p0 + u) * part_stride + d0));
                eb[u] = to_f32(act_load(row + (size_t)(p0 + u) * part_stride + d1));
            }
#pragma unroll
        for (int u = 0; u < 8; ++u)
            if (p0 + u < n_parts) {
                a += ea[u];
                b += eb[u];
            }
    }
    a += bias0;
    b += bias1;
    if (fi >= 0) {
        float s, c;
        rope_sincos(pos, f, f_lo, &s, &c);
        const float r0 = a * c - b * s, r1 = a * s + b * c;
        a = r0;
        b = r1;
    }
    if (head < H) {
        T *dst = q_out + (size_t)t * ldq + col;
        dst[d0] = from_f32<T>(a);
        dst[d1] = from_f32<T>(b);
        return;
    }
    if (page < 0 || page >= n_pages) {   // the host reserves pages first; never write outside the pool
        if (j == 0) atomicExch(status, 2);
        return;
    }
    const bool is_k = head < H + Hkv;
    const int g = is_k ? head - H : head - H - Hkv;
    T *dst = (is_k ? k_pages : v_pages) + (((size_t)page * Hkv + g) * page_size + (size_t)(pos % page_size)) * D;
    dst[d0] = from_f32<T>(a);
    dst[d1] = from_f32<T>(b);
}


// The same for many tokens at once (prompts), bfloat16 in and out, one part: a block per token.
// The token's cosines and sines are computed once and shared by all its heads, and a work unit
// is 16 bytes (8 elements) of one head, or for the "half" pairing the two 16-byte runs that
// hold 8 pairs, so that loads and stores are as wide as the hardware takes.  The arithmetic of
// one pair is that of the kernel above.
constexpr int WIDE_THREADS = 128;
constexpr int WIDE_MAX_ROT = 512;
__global__ void __launch_bounds__(WIDE_THREADS) rope_kv_write_wide_kernel(
    const __nv_bfloat16 *__restrict__ src, int lds, const float *__restrict__ bias, __nv_bfloat16 *__restrict__ q_out, int ldq,
    const int *__restrict__ positions, const int *__restrict__ seq_of_token, const int *__restrict__ block_table, int max_blocks,
    const float *__restrict__ inv_freq, const float *__restrict__ inv_freq_lo, int n_rot, int pairing, __nv_bfloat16 *__restrict__ k_pages,
    __nv_bfloat16 *__restrict__ v_pages, int n_pages, int page_size, int H, int Hkv, int D, int write_kv, int *__restrict__ status) {
    pdl_trigger();
    pdl_wait();
    __shared__ float2 cs[WIDE_MAX_ROT / 2];      // (cos, sin) of pair i
    const int t = blockIdx.x, tid = threadIdx.x;
    const int pos = positions[t];
    const int half_rot = n_rot / 2;
    for (int i = tid; i < half_rot; i += WIDE_THREADS) {
        float sn, c;
        rope_sincos(pos, inv_freq[i], inv_freq_lo ? inv_freq_lo[i] : 0.f, &sn, &c);
        cs[i] = make_float2(c, sn);
    }
    // where this token's k and v go
    int page = -1;
    if (write_kv) {
        const int seq = seq_of_token[t];
        const int blk = pos / page_size;
        if (pos >= 0 && blk < max_blocks) page = block_table[(size_t)seq * max_blocks + blk];
        if (page < 0 || page >= n_pages) {   // the host reserves pages first; never write outside the pool
            if (tid == 0) atomicExch(status, 2);
            page = -1;
        }
    }
    __syncthreads();
    const int rot_units = pairing ? n_rot / 8 : n_rot / 16;     // units of a rotated head that turn
    const int copy_units = (D - n_rot) / 8;                     // and those that pass through
    const int units_qk = rot_units + copy_units, units_v = D / 8;
    const int n_qk = write_kv ? H + Hkv : H;
    const int total = n_qk * units_qk + (write_kv ? Hkv * units_v : 0);
    const __nv_bfloat16 *row = src + (size_t)t * lds;
    for (int u = tid; u < total; u += WIDE_THREADS) {
        int head, unit;
        bool is_v = false;
        if (u < n_qk * units_qk) {
            head = u / units_qk;
            unit = u - head * units_qk;
        } else {
            const int w = u - n_qk * units_qk;
            head = H + Hkv + w / units_v;
            unit = w - (w / units_v) * units_v;
            is_v = true;
        }
        const size_t col = (size_t)head * D;
        __nv_bfloat16 *dst;
        if (head < H) {
            dst = q_out + (size_t)t * ldq + col;
        } else {
            if (page < 0) continue;
            const int g = is_v ? head - H - Hkv : head - H;
            dst = (is_v ? v_pages : k_pages) + (((size_t)page * Hkv + g) * page_size + (size_t)(pos % page_size)) * D;
        }
        if (is_v || unit >= rot_units) {
            // 8 elements that do not turn
            const int d = is_v ? unit * 8 : n_rot + (unit - rot_units) * 8;
            uint4 raw = act_load(reinterpret_cast<const uint4 *>(row + col + d));
            if (bias) {
                __nv_bfloat16 *e = reinterpret_cast<__nv_bfloat16 *>(&raw);
#pragma unroll
                for (int j = 0; j < 8; ++j) e[j] = __float2bfloat16_rn(__bfloat162float(e[j]) + bias[col + d + j]);
            }
            *reinterpret_cast<uint4 *>(dst + d) = raw;
        } else if (pairing) {
            // adjacent pairs: 8 elements = pairs 4 unit .. 4 unit + 3
            const int d = unit * 8;
            uint4 raw = act_load(reinterpret_cast<const uint4 *>(row + col + d));
            __nv_bfloat16 *e = reinterpret_cast<__nv_bfloat16 *>(&raw);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float a = __bfloat162float(e[2 * j]), b = __bfloat162float(e[2 * j + 1]);
                if (bias) {
                    a += bias[col + d + 2 * j];
                    b += bias[col + d + 2 * j + 1];
                }
                const float2 f = cs[unit * 4 + j];
                e[2 * j] = __float2bfloat16_rn(a * f.x - b * f.y);
                e[2 * j + 1] = __float2bfloat16_rn(a * f.y + b * f.x);
            }
            *reinterpret_cast<uint4 *>(dst + d) = raw;
        } else {
            // half pairs: elements 8 unit .. 8 unit + 7 with their partners n_rot / 2 further
            const int d0 = unit * 8, d1 = d0 + half_rot;
            uint4 ra = act_load(reinterpret_cast<const uint4 *>(row + col + d0));
            uint4 rb = act_load(reinterpret_cast<const uint4 *>(row + col + d1));
            __nv_bfloat16 *ea = reinterpret_cast<__nv_bfloat16 *>(&ra), *eb = reinterpret_cast<__nv_bfloat16 *>(&rb);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                float a = __bfloat162float(ea[j]), b = __bfloat162float(eb[j]);
                if (bias) {
                    a += bias[col + d0 + j];
                    b += bias[col + d1 + j];
                }
                const float2 f = cs[d0 + j];
                ea[j] = __float2bfloat16_rn(a * f.x - b * f.y);
                eb[j] = __float2bfloat16_rn(a * f.y + b * f.x);
            }
            *reinterpret_cast<uint4 *>(dst + d0) = ra;
            *reinterpret_cast<uint4 *>(dst + d1) = rb;
        }
    }
}

// Whether the wide kernel can take this call: 16-byte runs everywhere.
inline bool wide_ok(const void *src, int lds, const void *q_out, int ldq, const void *k_pages, const void *v_pages, int n_rot, int pairing,
                    int D, int n_tokens) {
    if (n_tokens < 32 || n_rot > WIDE_MAX_ROT) return false;
    if (D % 8 || lds % 8 || ldq % 8 || n_rot % (pairing ? 8 : 16)) return false;
    return (((uintptr_t)src | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15) == 0;
}

template <typename TS, typename T>
int launch(const void *src, int lds, int n_parts, long long part_stride, const float *bias, void *q_out, int ldq, const int *positions,
           const int *seq_of_token, const int *block_table, int max_blocks, const float *inv_freq, const float *inv_freq_lo, int n_rot, int pairing,
           void *k_pages, void *v_pages, int n_pages, int page_size, int n_tokens, int H, int Hkv, int D, int write_kv, int *status,
           cudaStream_t stream) {
    const int items = (write_kv ? H + 2 * Hkv : H) * (D / 2);
    dim3 grid(n_tokens, (items + ITEMS - 1) / ITEMS);
    lgml_launch(rope_kv_write_kernel<TS, T>, grid, ITEMS, 0, stream, (const TS *)src, lds, n_parts, part_stride, bias, (T *)q_out, ldq, positions,
                                                            seq_of_token, block_table, max_blocks, inv_freq, inv_freq_lo, n_rot, pairing, (T *)k_pages,
                                                            (T *)v_pages, n_pages, page_size, H, Hkv, D, write_kv, status);
    return lgml_launch_status("rope_kv_write");
}
// ---------------------------------------------------------------------------------------------
// conv_rope_store: q and k pass a short causal convolution over time per channel, the values are
// the convolved keys as they are (their first Dv entries), then q and k turn by their positions
// (pairs (i, i + n_rot / 2) of the first n_rot entries; cos and sin times `mag`), k and v go to
// their cells, q to its buffer.
//   proj float32 [n, ldp]: q at column 0 (H D), k behind it (G D); wT float32 [taps, (H + G) D] (row j weighs the
//   input taps - 1 - j tokens back); state: per slot (taps - 1) x (H + G) D floats, the oldest input first.
// One work item = one rotated pair, or one entry past n_rot, of one head of one token.  The tokens that reach back
// before the step's first token of their request are all computed by the item of that first token, which then
// writes the slot (no other item touches its floats there).
constexpr int CONV_MAX_TAPS = 8;

template <int V> struct CrsVec;
template <> struct CrsVec<1> {
    static __device__ __forceinline__ void load(const float *p, float (&v)[1]) { v[0] = act_load(p); }
    static __device__ __forceinline__ void load_w(const float *p, float (&v)[1]) { v[0] = __ldg(p); }
    static __device__ __forceinline__ void store(float *p, const float (&v)[1]) { p[0] = v[0]; }
    static __device__ __forceinline__ void store(__nv_bfloat16 *p, const float (&v)[1]) { p[0] = __float2bfloat16_rn(v[0]); }
};
template <> struct CrsVec<4> {
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

// V: neighbouring pairs (or unrotated entries) a work item takes: 4 when sizes, strides and addresses allow 16-byte
// loads and 8-byte stores, else 1.
template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(ITEMS) conv_rope_store_kernel(
    const float *__restrict__ proj, int ldp, const float *__restrict__ wT, float *__restrict__ state, long long state_ld, int taps_rt,
    T *__restrict__ q_out, int ldq, const int *__restrict__ positions, const int *__restrict__ seq_of_token, const int *__restrict__ seq_start,
    const int *__restrict__ slots, const int *__restrict__ block_table, int max_blocks, const float *__restrict__ inv_freq,
    const float *__restrict__ inv_freq_lo, float mag, int n_rot, T *__restrict__ k_pages, T *__restrict__ v_pages, int n_pages, int page_size,
    int H, int G, int D, int Dv, int write_kv, int *__restrict__ status, int n_tokens, int tpt) {
    pdl_trigger();
    pdl_wait();
    using X = CrsVec<V>;
    const int taps = TAPS > 0 ? TAPS : taps_rt;
    constexpr int MT = TAPS > 0 ? TAPS : CONV_MAX_TAPS;      // TAPS > 0: the taps at compile time
    constexpr int RUN = 4;      // tokens an item takes in a row when a step has many (tpt = RUN): a projected row is then read once for RUN results
    const int half_rot = n_rot / 2, iph = (half_rot + (D - n_rot)) / V;
    const int n_heads = write_kv ? H + G : H;
    const int item = blockIdx.y * ITEMS + threadIdx.x;
    if (item >= n_heads * iph) return;
    const int head = item / iph, j = (item - head * iph) * V;
    const int back = taps - 1;
    const int tA = blockIdx.x * tpt, tB = min(tA + tpt, n_tokens);
    int s = seq_of_token[tA];
    const int d0 = j < half_rot ? j : n_rot + (j - half_rot);
    const int d1 = j < half_rot ? j + half_rot : -1;
    const bool two = d1 >= 0;
    float f[V], f_lo[V];
#pragma unroll
    for (int e = 0; e < V; ++e) f[e] = two ? inv_freq[j + e] : 0.f, f_lo[e] = (two && inv_freq_lo) ? inv_freq_lo[j + e] : 0.f;
    const int C = (H + G) * D;
    const int c0 = head * D + d0, c1 = head * D + (two ? d1 : d0);
    float w0[MT][V], w1[MT][V];
#pragma unroll
    for (int k = 0; k < MT; ++k)
        if (k < taps) X::load_w(wT + (size_t)k * C + c0, w0[k]), X::load_w(wT + (size_t)k * C + c1, w1[k]);

    auto emit = [&](int tt, const float (&a)[V], const float (&b)[V]) {
        const int pos = positions[tt];
        float ra[V], rb[V];
#pragma unroll
        for (int e = 0; e < V; ++e) {
            ra[e] = a[e], rb[e] = b[e];
            if (two) {
                float sn, cs;
                rope_sincos(pos, f[e], f_lo[e], &sn, &cs);
                sn *= mag, cs *= mag;
                ra[e] = a[e] * cs - b[e] * sn;
                rb[e] = b[e] * cs + a[e] * sn;
            }
        }
        if (head < H) {
            T *qr = q_out + (size_t)tt * ldq + (size_t)head * D;
            X::store(qr + d0, ra);
            if (two) X::store(qr + d1, rb);
            return;
        }
        const int g = head - H;
        const int blk = pos / page_size;
        int page = -1;
        if (pos >= 0 && blk < max_blocks) page = block_table[(size_t)s * max_blocks + blk];
        if (page < 0 || page >= n_pages) {       // the host reserves pages first; never write outside the pool
            if (j == 0) atomicExch(status, 2);
            return;
        }
        const size_t cell = ((size_t)page * G + g) * page_size + (size_t)(pos % page_size);
        X::store(k_pages + cell * D + d0, ra);
        if (two) X::store(k_pages + cell * D + d1, rb);
        if (d0 < Dv) X::store(v_pages + cell * Dv + d0, a);          // (with V = 4 the value size is a multiple of 4: a group lies inside or outside)
        if (two && d1 < Dv) X::store(v_pages + cell * Dv + d1, b);
    };

    if (TAPS > 0 && tpt == RUN && tB - tA == RUN && s == seq_of_token[tA + RUN - 1] && tA - seq_start[s] >= back) {
        // RUN tokens of one request, none of which reaches into the slot: a window of back + RUN projected rows
        float in0[MT - 1 + RUN][V], in1[MT - 1 + RUN][V];
#pragma unroll
        for (int r = 0; r < MT - 1 + RUN; ++r) {
            const float *row = proj + (size_t)(tA - back + r) * ldp;
            X::load(row + c0, in0[r]);
            if (two) X::load(row + c1, in1[r]);
        }
#pragma unroll
        for (int q = 0; q < RUN; ++q) {
            float a[V], b[V];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                a[e] = b[e] = 0.f;
#pragma unroll
                for (int k = 0; k < MT; ++k) {
                    a[e] = fmaf(w0[k][e], in0[q + k][e], a[e]);
                    if (two) b[e] = fmaf(w1[k][e], in1[q + k][e], b[e]);
                }
            }
            emit(tA + q, a, b);
        }
        return;
    }
    for (int t = tA; t < tB; ++t) {
    s = seq_of_token[t];
    const int t0 = seq_start[s];
    const int i = t - t0;
    if (i > 0 && i < back) continue;
    if (i >= back) {
        float a[V], b[V];
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = b[e] = 0.f;
#pragma unroll
        for (int k = 0; k < MT; ++k) {
            if (k < taps) {
                const float *row = proj + (size_t)(t - back + k) * ldp;
                float u0[V], u1[V];
                X::load(row + c0, u0);
                if (two) X::load(row + c1, u1);
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    a[e] = fmaf(w0[k][e], u0[e], a[e]);
                    if (two) b[e] = fmaf(w1[k][e], u1[e], b[e]);
                }
            }
        }
        emit(t, a, b);
        continue;
    }
    const int n_s = seq_start[s + 1] - t0;
    float *st = state + (size_t)slots[s] * state_ld;
    float old0[MT][V], old1[MT][V];
#pragma unroll
    for (int r = 0; r < MT; ++r) {
        if (r < back) {
            X::load(st + (size_t)r * C + c0, old0[r]);
            if (two) X::load(st + (size_t)r * C + c1, old1[r]);
        }
    }
    const int first = n_s < back ? n_s : back;
    for (int kk = 0; kk < first; ++kk) {
        float a[V], b[V];
#pragma unroll
        for (int e = 0; e < V; ++e) a[e] = b[e] = 0.f;
#pragma unroll
        for (int k = 0; k < MT; ++k) {
            if (k < taps) {
                const int rel = kk - back + k;
                float u0[V], u1[V];
#pragma unroll
                for (int e = 0; e < V; ++e) u0[e] = u1[e] = 0.f;
                if (rel >= 0) {
                    X::load(proj + (size_t)(t0 + rel) * ldp + c0, u0);
                    if (two) X::load(proj + (size_t)(t0 + rel) * ldp + c1, u1);
                } else {
#pragma unroll
                    for (int r = 0; r < MT; ++r)
                        if (r == back + rel) {
#pragma unroll
                            for (int e = 0; e < V; ++e) u0[e] = old0[r][e], u1[e] = two ? old1[r][e] : 0.f;
                        }
                }
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    a[e] = fmaf(w0[k][e], u0[e], a[e]);
                    if (two) b[e] = fmaf(w1[k][e], u1[e], b[e]);
                }
            }
        }
        emit(t0 + kk, a, b);
    }
#pragma unroll
    for (int r = 0; r < MT; ++r) {
        if (r < back) {
            const int rel = n_s - back + r;
            float v0[V], v1[V];
#pragma unroll
            for (int e = 0; e < V; ++e) v0[e] = v1[e] = 0.f;
            if (rel >= 0) {
                X::load(proj + (size_t)(t0 + rel) * ldp + c0, v0);
                if (two) X::load(proj + (size_t)(t0 + rel) * ldp + c1, v1);
            } else {
#pragma unroll
                for (int q = 0; q < MT; ++q)
                    if (q == back + rel) {
#pragma unroll
                        for (int e = 0; e < V; ++e) v0[e] = old0[q][e], v1[e] = two ? old1[q][e] : 0.f;
                    }
            }
            X::store(st + (size_t)r * C + c0, v0);
            if (two) X::store(st + (size_t)r * C + c1, v1);
        }
    }
    }
}
// ---------------------------------------------------------------------------------------------
// norm_rope_store: q and k are normed head by head (over the root mean square of the head's D entries, times a weight of
// size D shared by the heads; weight null: no norm), then turn by their positions (pairs (i, i + n_rot / 2) of the first
// n_rot entries); k and v (times v_scale) go to their cells, q to its buffer.
//   proj float32 [n, ldp]: q at column 0 (H D), k behind it (G D), v behind that (G Dv).
// Block: a token and a share of its heads; a warp takes one head at a time through a row of shared memory.  The cosines
// and sines of the token's position are computed once per block.
constexpr int NRS_WARPS = 4;

template <typename T, int V>
__global__ void __launch_bounds__(NRS_WARPS * 32) norm_rope_store_kernel(
    const float *__restrict__ proj, int ldp, const float *__restrict__ q_w, const float *__restrict__ k_w, float eps, T *__restrict__ q_out, int ldq,
    const int *__restrict__ positions, const int *__restrict__ seq_of_token, const int *__restrict__ block_table, int max_blocks,
    const float *__restrict__ inv_freq, const float *__restrict__ inv_freq_lo, int n_rot, T *__restrict__ k_pages, T *__restrict__ v_pages, int n_pages,
    int page_size, int H, int G, int D, int Dv, float v_scale, int write_kv, int *__restrict__ status) {
    pdl_trigger();
    pdl_wait();
    using X = CrsVec<V>;
    extern __shared__ __align__(16) float nrs[];
    const int half = n_rot / 2, DS = (max(D, Dv) + 3) & ~3;
    float *cosv = nrs, *sinv = nrs + half, *rows = nrs + ((n_rot + 3) & ~3);
    const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int pos = positions[t];
    for (int i = threadIdx.x; i < half; i += NRS_WARPS * 32) rope_sincos(pos, inv_freq[i], inv_freq_lo ? inv_freq_lo[i] : 0.f, sinv + i, cosv + i);
    int page = -1;
    if (write_kv) {
        const int blk = pos / page_size;
        if (pos >= 0 && blk < max_blocks) page = block_table[(size_t)seq_of_token[t] * max_blocks + blk];
        if (page < 0 || page >= n_pages) {       // the host reserves pages first; never write outside the pool
            if (threadIdx.x == 0 && blockIdx.y == 0) atomicExch(status, 2);
            page = -1;
        }
    }
    __syncthreads();
    float *buf = rows + (size_t)warp * DS;
    const float *row = proj + (size_t)t * ldp;
    const int n_heads = write_kv ? H + 2 * G : H;
    for (int head = blockIdx.y * NRS_WARPS + warp; head < n_heads; head += gridDim.y * NRS_WARPS) {
        const size_t cell_row = (size_t)(pos % page_size);
        if (head >= H + G) {
            if (page < 0) continue;
            const int g = head - H - G;
            const float *src = row + (size_t)(H + G) * D + (size_t)g * Dv;
            T *dst = v_pages + (((size_t)page * G + g) * page_size + cell_row) * Dv;
            for (int d = lane * V; d < Dv; d += 32 * V) {
                float v[V];
                X::load(src + d, v);
#pragma unroll
                for (int e = 0; e < V; ++e) v[e] *= v_scale;
                X::store(dst + d, v);
            }
            continue;
        }
        const bool is_q = head < H;
        const float *w = is_q ? q_w : k_w, *src = row + (size_t)head * D;
        float ss = 0.f;
        for (int d = lane * V; d < D; d += 32 * V) {
            float v[V];
            X::load(src + d, v);
#pragma unroll
            for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss), buf[d + e] = v[e];
        }
        float inv = 1.f;
        if (w != nullptr) {
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)D + eps);
            for (int d = lane * V; d < D; d += 32 * V) {
                float g[V];
                X::load_w(w + d, g);
#pragma unroll
                for (int e = 0; e < V; ++e) buf[d + e] = buf[d + e] * inv * g[e];
            }
        }
        __syncwarp();
        T *dst = is_q ? q_out + (size_t)t * ldq + (size_t)head * D
                      : (page >= 0 ? k_pages + (((size_t)page * G + (head - H)) * page_size + cell_row) * D : nullptr);
        if (dst != nullptr)
            for (int d = lane * V; d < D; d += 32 * V) {
                float y[V];
#pragma unroll
                for (int e = 0; e < V; ++e) {
                    const int i = d + e;
                    y[e] = buf[i];
                    if (i < half) y[e] = buf[i] * cosv[i] - buf[i + half] * sinv[i];
                    else if (i < n_rot) y[e] = buf[i] * cosv[i - half] + buf[i - half] * sinv[i - half];
                }
                X::store(dst + d, y);
            }
        __syncwarp();
    }
}
}  // namespace

// src: [n_parts][n_tokens][(H + 2 Hkv) D] of src_dtype (row stride lds, part_stride elements between
// parts; n_parts > 1 only with float32).  q_out (dtype, row stride ldq) may be src itself when
// n_parts == 1 and the types agree (rotation in place).  The cache has type `dtype`.
// inv_freq: n_rot / 2 frequencies; inv_freq_lo: what float32 lost of each (table - (float)table), or null.
LGML_API int lgml_rope_kv_write(const void *src, int src_dtype, int lds, int n_parts, long long part_stride, const float *bias,
                                void *q_out, int dtype, int ldq, const int *positions, const int *seq_of_token,
                                const int *block_table, int max_blocks, const float *inv_freq, const float *inv_freq_lo, int n_rot,
                                int pairing, void *k_pages, void *v_pages, int n_pages, int page_size, int n_tokens, int H, int Hkv, int D,
                                int write_kv, int *status, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && H > 0 && Hkv > 0 && D > 0 && page_size > 0 && max_blocks > 0, "rope_kv_write: bad sizes");
    LGML_REQUIRE(D % 2 == 0, "rope_kv_write: head_dim %d must be even", D);
    LGML_REQUIRE(n_rot >= 0 && n_rot <= D && n_rot % 2 == 0, "rope_kv_write: n_rot %d must be even and at most head_dim %d", n_rot, D);
    LGML_REQUIRE(lds >= (H + 2 * Hkv) * D, "rope_kv_write: row stride %d is below (H + 2 Hkv) D = %d", lds, (H + 2 * Hkv) * D);
    LGML_REQUIRE(ldq >= H * D, "rope_kv_write: q row stride %d is below H D = %d", ldq, H * D);
    LGML_REQUIRE(pairing == 0 || pairing == 1, "rope_kv_write: unknown pairing %d", pairing);
    LGML_REQUIRE(n_parts >= 1 && (n_parts == 1 || src_dtype == LGML_F32), "rope_kv_write: partial sums are float32");
    if (n_tokens == 0) return 0;
#define ARGS src, lds, n_parts, part_stride, bias, q_out, ldq, positions, seq_of_token, block_table, max_blocks, inv_freq, inv_freq_lo, n_rot, pairing, \
             k_pages, v_pages, n_pages, page_size, n_tokens, H, Hkv, D, write_kv, status, stream
    if (src_dtype == LGML_F32 && dtype == LGML_F32) return launch<float, float>(ARGS);
    if (src_dtype == LGML_F32 && dtype == LGML_BF16) return launch<float, __nv_bfloat16>(ARGS);
    if (src_dtype == LGML_BF16 && dtype == LGML_BF16) {
        if (n_parts == 1 && wide_ok(src, lds, q_out, ldq, k_pages, v_pages, n_rot, pairing, D, n_tokens)) {
            lgml_launch(rope_kv_write_wide_kernel, dim3(n_tokens), WIDE_THREADS, 0, stream, (const __nv_bfloat16 *)src, lds, bias,
                        (__nv_bfloat16 *)q_out, ldq, positions, seq_of_token, block_table, max_blocks, inv_freq, inv_freq_lo, n_rot, pairing,
                        (__nv_bfloat16 *)k_pages, (__nv_bfloat16 *)v_pages, n_pages, page_size, H, Hkv, D, write_kv, status);
            return lgml_launch_status("rope_kv_write");
        }
        return launch<__nv_bfloat16, __nv_bfloat16>(ARGS);
    }
#undef ARGS
    LGML_FAIL("rope_kv_write: unsupported types (source %d, output %d)", src_dtype, dtype);
}


// q and k through a short convolution (taps >= 1; 1: none, w is then one row), the values are the convolved keys'
// first Dv entries, rotation of the first n_rot entries of q and k with cos and sin times mag; see the kernel.
LGML_API int lgml_conv_rope_store(const float *proj, int ldp, const float *wT, float *state, long long state_ld, int taps, void *q_out, int dtype,
                                  int ldq, const int *positions, const int *seq_of_token, const int *seq_start, const int *slots,
                                  const int *block_table, int max_blocks, const float *inv_freq, const float *inv_freq_lo, float mag, int n_rot,
                                  void *k_pages, void *v_pages, int n_pages, int page_size, int n_tokens, int H, int G, int D, int Dv, int write_kv,
                                  int *status, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && H > 0 && G > 0 && D > 0 && Dv > 0 && Dv <= D && page_size > 0 && max_blocks > 0, "conv_rope_store: bad sizes");
    LGML_REQUIRE(n_rot >= 0 && n_rot <= D && n_rot % 2 == 0, "conv_rope_store: n_rot %d must be even and at most the head size %d", n_rot, D);
    LGML_REQUIRE(taps >= 1 && taps <= CONV_MAX_TAPS, "conv_rope_store: 1 to %d taps, not %d", CONV_MAX_TAPS, taps);
    LGML_REQUIRE(taps == 1 || (state != nullptr && state_ld >= (long long)(taps - 1) * (H + G) * D), "conv_rope_store: the state's rows are too short");
    LGML_REQUIRE(ldp >= (H + G) * D && ldq >= H * D, "conv_rope_store: rows too short");
    if (n_tokens == 0) return 0;
    const bool vec = (n_rot / 2) % 4 == 0 && (D - n_rot) % 4 == 0 && Dv % 4 == 0 && ldp % 4 == 0 && ldq % 4 == 0 && state_ld % 4 == 0 &&
                     ((((uintptr_t)proj | (uintptr_t)wT | (uintptr_t)state | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15) == 0);
    const int iph = (n_rot / 2 + (D - n_rot)) / (vec ? 4 : 1);
    const int items = (write_kv ? H + G : H) * iph;
    const int tpt = n_tokens >= 256 ? 4 : 1;          // many tokens: an item takes four in a row
    dim3 grid((n_tokens + tpt - 1) / tpt, (items + ITEMS - 1) / ITEMS);
#define LGML_CRS_T(T, V, TP) lgml_launch(conv_rope_store_kernel<T, V, TP>, grid, ITEMS, 0, stream, proj, ldp, wT, state, state_ld, taps, (T *)q_out, ldq, positions, \
                                   seq_of_token, seq_start, slots, block_table, max_blocks, inv_freq, inv_freq_lo, mag, n_rot, (T *)k_pages, (T *)v_pages, \
                                   n_pages, page_size, H, G, D, Dv, write_kv, status, n_tokens, tpt)
#define LGML_CRS(T, V) \
    do { switch (taps) { case 2: LGML_CRS_T(T, V, 2); break; case 3: LGML_CRS_T(T, V, 3); break; case 4: LGML_CRS_T(T, V, 4); break; default: LGML_CRS_T(T, V, 0); } } while (0)
    if (dtype == LGML_F32) { if (vec) LGML_CRS(float, 4); else LGML_CRS(float, 1); }
    else if (dtype == LGML_BF16) { if (vec) LGML_CRS(__nv_bfloat16, 4); else LGML_CRS(__nv_bfloat16, 1); }
    else LGML_FAIL("conv_rope_store: unknown type %d", dtype);
#undef LGML_CRS
#undef LGML_CRS_T
    return lgml_launch_status("conv_rope_store");
}

// The norm per head, the turn and the cache write; see the kernel.  q_w / k_w: float32 [D] or null.
LGML_API int lgml_norm_rope_store(const float *proj, int ldp, const float *q_w, const float *k_w, float eps, void *q_out, int dtype, int ldq,
                                  const int *positions, const int *seq_of_token, const int *block_table, int max_blocks, const float *inv_freq,
                                  const float *inv_freq_lo, int n_rot, void *k_pages, void *v_pages, int n_pages, int page_size, int n_tokens, int H, int G,
                                  int D, int Dv, float v_scale, int write_kv, int *status, cudaStream_t stream) {
    LGML_REQUIRE(n_tokens >= 0 && H > 0 && G > 0 && D > 0 && Dv > 0 && page_size > 0 && max_blocks > 0, "norm_rope_store: bad sizes");
    LGML_REQUIRE(n_rot >= 0 && n_rot <= D && n_rot % 2 == 0, "norm_rope_store: n_rot %d must be even and at most the head size %d", n_rot, D);
    LGML_REQUIRE(ldp >= (H + G) * D + G * Dv && ldq >= H * D, "norm_rope_store: rows too short");
    if (n_tokens == 0) return 0;
    const int DS = ((D > Dv ? D : Dv) + 3) & ~3;
    const size_t smem = sizeof(float) * (size_t)(((n_rot + 3) & ~3) + NRS_WARPS * DS);
    LGML_REQUIRE(smem <= 48 * 1024, "norm_rope_store: heads of %d and %d do not fit shared memory", D, Dv);
    const bool vec = D % 4 == 0 && Dv % 4 == 0 && ldp % 4 == 0 && ldq % 4 == 0 &&
                     ((((uintptr_t)proj | (uintptr_t)q_w | (uintptr_t)k_w | (uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & 15) == 0);
    // a token's heads go over several blocks while tokens alone do not fill the SMs
    const int n_heads = write_kv ? H + 2 * G : H;
    int splits = (n_heads + NRS_WARPS - 1) / NRS_WARPS;
    while (splits > 1 && (long long)n_tokens * splits > 148 * 16) splits = (splits + 1) / 2;
    dim3 grid(n_tokens, splits);
#define LGML_NRS(T, V) lgml_launch(norm_rope_store_kernel<T, V>, grid, NRS_WARPS * 32, smem, stream, proj, ldp, q_w, k_w, eps, (T *)q_out, ldq, positions, \
                                   seq_of_token, block_table, max_blocks, inv_freq, inv_freq_lo, n_rot, (T *)k_pages, (T *)v_pages, n_pages, page_size, H, G, \
                                   D, Dv, v_scale, write_kv, status)
    if (dtype == LGML_F32) { if (vec) LGML_NRS(float, 4); else LGML_NRS(float, 1); }
    else if (dtype == LGML_BF16) { if (vec) LGML_NRS(__nv_bfloat16, 4); else LGML_NRS(__nv_bfloat16, 1); }
    else LGML_FAIL("norm_rope_store: unknown type %d", dtype);
#undef LGML_NRS
    return lgml_launch_status("norm_rope_store");
}
