// Linear recurrences with one decay per head over many tokens, in chunks of 64 tokens (all float32, on FMA units):
//
//   delta rule      S <- a S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
//   matrix memory   S <- a S + b k v^T;                                o = S^T q        (optionally one more column whose v is 1)
//
// With G_i the sum of log a over a chunk's tokens 0 .. i and S0 the state ahead of the chunk, a chunk is a handful of
// small matrix products instead of 64 dependent steps:
//
//   M_ij = e^(G_i - G_j) (q_i . k_j) w_j   for j <= i       w: 1 (delta), b (memory)
//   A_ij = beta_i e^(G_i - G_j) (k_i . k_j) for j < i,      T = (1 + A)^-1 diag(beta)          (delta only)
//   U    = T (V - e^G K S0)  (delta),  V  (memory)
//   O    = e^G Q S0 + M U
//   S    = e^(G_last) S0 + K^T (e^(G_last - G) w U)
//
// Every exponent is at most 0 (decays are at most 1), so nothing overflows however strong the decay; the sums G are held in
// double precision, so a difference of two large ones keeps float32's precision.
//
//   chunk_prepare   per (chunk, key head): T, M and the row factors; chunks side by side, no state involved.  1 + A is
//                   lower triangular with ones on the diagonal: a thread solves one column of its inverse.
//   chunk_scan      per (request, head, group of columns): the chunks in order; the columns of S are independent of each
//                   other, so a block keeps its columns of S in shared memory and walks the chunks, with the next
//                   chunk's operands on their way (cp.async) while this one is computed
#include <math.h>

#include "common.cuh"

LGML_DEFINE_LAST_ERROR(lgml_chunk_scan)

namespace {
constexpr int CT = 64;              // tokens of a chunk
constexpr int LDC = CT + 4;         // floats between rows of a 64-wide matrix in shared memory
constexpr int PREP_THREADS = 256, SCAN_THREADS = 512;
constexpr int FAC = 2 * CT + 4;     // per (chunk, head): e^G (64), e^(G_last - G) w (64), e^(G_last), zeros

__device__ __forceinline__ void cp16(float *dst, const float *src, bool valid) {
    const int bytes = valid ? 16 : 0;           // 0: zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// two float32 products-and-sums in one instruction
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(*reinterpret_cast<uint64_t *>(&a)), "l"(*reinterpret_cast<uint64_t *>(&b)), "l"(*reinterpret_cast<uint64_t *>(&c)));
    return *reinterpret_cast<float2 *>(&d);
}

// nt rows of D floats (ld apart) into rows of LD floats; rows nt .. 63 become zeros
template <int THREADS>
__device__ __forceinline__ void stage_rows(float *dst, int LD, const float *src, long long ld, int nt, int D, int tid) {
    const int d4 = D / 4, di = THREADS / d4, dc = THREADS - di * d4;
    int i = tid / d4, c = tid - i * d4;
    while (i < CT) {                            // (one division per call: rows and columns then advance by steps)
        const bool ok = i < nt;
        cp16(dst + i * LD + c * 4, src + (ok ? (long long)i * ld : 0) + c * 4, ok);
        i += di, c += dc;
        if (c >= d4) c -= d4, ++i;
    }
}

struct PrepArgs {
    const float *q, *k;             // row t: q + t ldx + g D, k + t ldx + g D
    int ldx;
    const float *log_a, *w;         // row t: + t ldg + h lhg; w: beta (delta) or b (memory)
    int ldg, lhg;
    const int *pieces;              // [n_chunks][2]: first token, past the last
    float *T, *M, *fac;             // [n_chunks][H][64][64] (T: delta only), [n_chunks][H][FAC]
    int H, G, D;
};

// C_ij = sum_d a_i[d] b_j[d] for all i, j < 64 (rows LD apart), two left operands at once when A1 is given; a thread has the
// rows ti + 16 r and the columns tj + 16 c
template <int NA>
__device__ __forceinline__ void dots_64(const float *A0, const float *A1, const float *B, int LD, int D, int tid, float (&acc)[NA][4][4]) {
    const int ti = (tid & 7) | ((tid >> 4) & 8), tj = ((tid >> 3) & 3) | ((tid >> 3) & 12);
#pragma unroll
    for (int n = 0; n < NA; ++n)
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int c = 0; c < 4; ++c) acc[n][r][c] = 0.f;
    for (int d = 0; d < D; d += 4) {
        float4 b[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) b[c] = *reinterpret_cast<const float4 *>(B + (tj + 16 * c) * LD + d);
#pragma unroll
        for (int n = 0; n < NA; ++n)
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                const float4 a = *reinterpret_cast<const float4 *>((n ? A1 : A0) + (ti + 16 * r) * LD + d);
#pragma unroll
                for (int c = 0; c < 4; ++c)
                    acc[n][r][c] = fmaf(a.x, b[c].x, fmaf(a.y, b[c].y, fmaf(a.z, b[c].z, fmaf(a.w, b[c].w, acc[n][r][c]))));
            }
    }
}

template <bool DELTA>
__global__ void __launch_bounds__(PREP_THREADS) chunk_prepare_kernel(const PrepArgs p) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int D = p.D, LD = D + 4, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int c = blockIdx.x, g = blockIdx.y, per = p.H / p.G;
    const int t0 = p.pieces[2 * c], nt = p.pieces[2 * c + 1] - t0;
    float *Ks = sm, *Qs = Ks + CT * LD;
    __shared__ double Gs[2][CT];
    __shared__ float ws[2][CT];
    stage_rows<PREP_THREADS>(Ks, LD, p.k + (size_t)t0 * p.ldx + (size_t)g * D, p.ldx, nt, D, tid);
    stage_rows<PREP_THREADS>(Qs, LD, p.q + (size_t)t0 * p.ldx + (size_t)g * D, p.ldx, nt, D, tid);
    cp_commit();
    cp_wait<0>();
    __syncthreads();
    float acc[DELTA ? 2 : 1][4][4];
    dots_64<DELTA ? 2 : 1>(Qs, Ks, Ks, LD, D, tid, acc);
    __syncthreads();                            // K and Q have been read; their room holds the products from here on
    float *QK = sm, *KK = sm + CT * LDC, *As = KK + CT * LDC;         // As: two heads' A
    {
        const int ti = (tid & 7) | ((tid >> 4) & 8), tj = ((tid >> 3) & 3) | ((tid >> 3) & 12);
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int cc = 0; cc < 4; ++cc) {
                QK[(ti + 16 * r) * LDC + tj + 16 * cc] = acc[0][r][cc];
                if (DELTA) KK[(ti + 16 * r) * LDC + tj + 16 * cc] = acc[DELTA ? 1 : 0][r][cc];
            }
    }
    for (int h0 = 0; h0 < per; h0 += 2) {
        __syncthreads();                        // the products are there; the pair of heads before is done with Gs, ws, As
        if (warp < 2 && h0 + warp < per) {
            const int h = g * per + h0 + warp;
            double x[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int i = 2 * lane + u;
                const bool ok = i < nt;
                const size_t at = (size_t)(t0 + (ok ? i : 0)) * p.ldg + (size_t)h * p.lhg;
                x[u] = ok ? (double)act_load(p.log_a + at) : 0.0;
                ws[warp][i] = ok ? act_load(p.w + at) : 0.f;
            }
            double s = x[0] + x[1];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const double up = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += up;
            }
            const double last = __shfl_sync(0xffffffffu, s, 31);
            Gs[warp][2 * lane] = s - x[1];
            Gs[warp][2 * lane + 1] = s;
            float *f = p.fac + ((size_t)c * p.H + h) * FAC;
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int i = 2 * lane + u;
                const double Gi = u ? s : s - x[1];
                f[i] = i < nt ? expf((float)Gi) : 0.f;
                f[CT + i] = i < nt ? expf((float)(last - Gi)) * (DELTA ? 1.f : ws[warp][i]) : 0.f;
            }
            if (lane < 4) f[2 * CT + lane] = lane == 0 ? expf((float)last) : 0.f;
        }
        __syncthreads();
        const int nh = min(2, per - h0);
        for (int hh = 0; hh < nh; ++hh) {
            float *Mo = p.M + ((size_t)c * p.H + g * per + h0 + hh) * CT * CT;
            for (int e = tid; e < CT * CT; e += PREP_THREADS) {
                const int i = e >> 6, j = e & 63;
                float m = 0.f, a = 0.f;
                if (j <= i && i < nt) {
                    const float ex = expf((float)(Gs[hh][i] - Gs[hh][j]));
                    m = ex * QK[i * LDC + j] * (DELTA ? 1.f : ws[hh][j]);
                    if (DELTA && j < i) a = ws[hh][i] * ex * KK[i * LDC + j];
                }
                Mo[e] = m;
                if (DELTA) As[(hh * CT + i) * LDC + j] = a;
            }
        }
        if (DELTA) {
            __syncthreads();
            const int hh = tid >> 6, j = tid & 63;
            if (hh < nh) {
                // column j of (1 + A)^-1, top down: x_i = [i = j] - sum_{l < i} A_il x_l
                const float *A = As + hh * CT * LDC;
                const float beta = ws[hh][j];
                float *To = p.T + ((size_t)c * p.H + g * per + h0 + hh) * CT * CT + j;
                float x[CT];
#pragma unroll
                for (int i = 0; i < CT; ++i) {
                    float s4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                    for (int l = 0; l < i; l += 4) {
                        const float4 a = *reinterpret_cast<const float4 *>(A + i * LDC + l);
                        s4[0] = fmaf(a.x, x[l], s4[0]);
                        if (l + 1 < i) s4[1] = fmaf(a.y, x[l + 1], s4[1]);
                        if (l + 2 < i) s4[2] = fmaf(a.z, x[l + 2], s4[2]);
                        if (l + 3 < i) s4[3] = fmaf(a.w, x[l + 3], s4[3]);
                    }
                    x[i] = (i == j ? 1.f : 0.f) - ((s4[0] + s4[1]) + (s4[2] + s4[3]));
                    To[i * CT] = i < nt ? x[i] * beta : 0.f;       // (beta is 0 for columns past the last token)
                }
            }
        }
    }
}

struct ScanArgs {
    const float *q, *k, *v;         // row t: q + t ldx + g D, k + t ldx + g D, v + t ldx + h Pv
    int ldx;
    const float *T, *M, *fac;
    const int *pieces, *first_piece, *req;      // req[r]: the request's index in slots
    float *state;
    long long state_ld;
    int s_row, s_col;               // S(d, col) of a head at d s_row + col s_col
    const int *slots;
    float *o;                       // row t: o + t ldo + h P
    int ldo;
    int H, G, D, Pv, P;             // P columns of S, the first Pv of them from v, the rest written with v = 1
    int v_vec;
};

// own[r][c] = A[row r] . Bt[col c], each lane over its share of the contraction, then added up over the SPLIT lanes that share the
// tile: a thread ends with TC / SPLIT of the tile's columns.  A thread's rows are rg + (64 / RT) r.
template <int RT, int TC, int SPLIT> struct Tile {
    static constexpr int GROUPS = CT / RT;          // row groups
    static constexpr int OWN = TC / SPLIT;
    static_assert(SPLIT == 4 && TC % 4 == 0, "four lanes share a tile");
    int rg, cg, sp;
    __device__ __forceinline__ explicit Tile(int i) {
        sp = (i >> 3) & 3;
        const int rest = i >> 5;
        rg = (i & 7) + 8 * (rest % (GROUPS / 8));
        cg = rest / (GROUPS / 8);
    }
    __device__ __forceinline__ int row(int r) const { return rg + GROUPS * r; }
    __device__ __forceinline__ int col(int c) const { return cg * TC + (sp >> 1) * (TC / 2) + (sp & 1) * (TC / 4) + c; }      // the thread's c-th own column
    __device__ __forceinline__ void run(const float *A, int lda, const float *Bt, int ldb, int quads, float (&own)[RT][OWN]) const {
        float2 acc2[RT][TC];                         // even and odd places of the contraction
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int c = 0; c < TC; ++c) acc2[r][c] = make_float2(0.f, 0.f);
        const float *b0 = Bt + (size_t)(cg * TC) * ldb, *a0 = A + rg * lda;
        for (int kq = sp; kq < quads; kq += SPLIT) {
            float4 a[RT];
#pragma unroll
            for (int r = 0; r < RT; ++r) a[r] = *reinterpret_cast<const float4 *>(a0 + GROUPS * r * lda + kq * 4);
#pragma unroll
            for (int c = 0; c < TC; ++c) {
                const float4 b = *reinterpret_cast<const float4 *>(b0 + c * ldb + kq * 4);
#pragma unroll
                for (int r = 0; r < RT; ++r)
                    acc2[r][c] = fma2(make_float2(a[r].x, a[r].y), make_float2(b.x, b.y), fma2(make_float2(a[r].z, a[r].w), make_float2(b.z, b.w), acc2[r][c]));
            }
        }
        float acc[RT][TC];
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int c = 0; c < TC; ++c) acc[r][c] = acc2[r][c].x + acc2[r][c].y;
        constexpr int H1 = TC / 2, H2 = TC / 4;
        const bool up1 = sp >> 1, up2 = sp & 1;
#pragma unroll
        for (int r = 0; r < RT; ++r) {
            float half[H1];
#pragma unroll
            for (int c = 0; c < H1; ++c) {
                const float send = up1 ? acc[r][c] : acc[r][c + H1], keep = up1 ? acc[r][c + H1] : acc[r][c];
                half[c] = keep + __shfl_xor_sync(0xffffffffu, send, 16);
            }
#pragma unroll
            for (int c = 0; c < H2; ++c) {
                const float send = up2 ? half[c] : half[c + H2], keep = up2 ? half[c + H2] : half[c];
                own[r][c] = keep + __shfl_xor_sync(0xffffffffu, send, 8);
            }
        }
    }
};

template <bool DELTA, int CB>
__global__ void __launch_bounds__(SCAN_THREADS, 1) chunk_scan_kernel(const ScanArgs p) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int D = p.D, LD = D + 4, LV = CB + 4, tid = threadIdx.x;
    float *Kb = sm;                              // two buffers of [64][LD]
    float *Qs = Kb + 2 * CT * LD;
    float *Ms = Qs + CT * LD;                    // [64][LDC]
    float *Ts = Ms + CT * LDC;                   // [64][LDC] (delta)
    float *Vs = Ts + (DELTA ? CT * LDC : 0);     // [64][LV]
    float *Fs = Vs + CT * LV;                    // FAC factors, two buffers
    float *Ot = Fs + 2 * FAC;                    // [CB][LDC]: e^G Q S0, then O, a row a column of S
    float *Xt = Ot + CB * LDC;                   // [CB][LDC]: V - e^G K S0 (delta)
    float *Ut = Xt + (DELTA ? CB * LDC : 0);     // [CB][LDC]: U
    float *Wt = Ut + CB * LDC;                   // [CB][LDC]: e^(G_last - G) w U
    float *St = Wt + CB * LDC;                   // [CB][LD]: S, a row a column
    const int r = blockIdx.z, h = blockIdx.y, g = h / (p.H / p.G), col0 = blockIdx.x * CB;
    const int c0 = p.first_piece[r], c1 = p.first_piece[r + 1];
    float *S_base = p.state + (size_t)p.slots[p.req[r]] * p.state_ld + (size_t)h * D * p.P;
    for (int e = tid; e < D * CB; e += SCAN_THREADS) {
        // (neighbouring threads along the direction in which the state is contiguous)
        const int d = p.s_row == 1 ? e % D : e / CB, c = p.s_row == 1 ? e / D : e % CB;
        St[c * LD + d] = col0 + c < p.P ? act_load(S_base + (size_t)d * p.s_row + (size_t)(col0 + c) * p.s_col) : 0.f;
    }
    auto stage_k = [&](int c) {
        if (c < c1) {
            const int t0 = p.pieces[2 * c], nt = p.pieces[2 * c + 1] - t0;
            stage_rows<SCAN_THREADS>(Kb + ((c - c0) & 1) * CT * LD, LD, p.k + (size_t)t0 * p.ldx + (size_t)g * D, p.ldx, nt, D, tid);
            const float *f = p.fac + ((size_t)c * p.H + h) * FAC;
            if (tid < FAC / 4) cp16(Fs + ((c - c0) & 1) * FAC + tid * 4, f + tid * 4, true);
        }
        cp_commit();
    };
    auto stage_qv = [&](int c) {
        if (c < c1) {
            const int t0 = p.pieces[2 * c], nt = p.pieces[2 * c + 1] - t0;
            stage_rows<SCAN_THREADS>(Qs, LD, p.q + (size_t)t0 * p.ldx + (size_t)g * D, p.ldx, nt, D, tid);
            const float *v = p.v + (size_t)t0 * p.ldx + (size_t)h * p.Pv + col0;
            if (p.v_vec && col0 + CB <= p.Pv) {
                for (int e = tid; e < CT * (CB / 4); e += SCAN_THREADS) {
                    const int i = e / (CB / 4), cc = (e - i * (CB / 4)) * 4;
                    const bool ok = i < nt;
                    cp16(Vs + i * LV + cc, v + (ok ? (size_t)i * p.ldx : 0) + cc, ok);
                }
            } else {
                for (int e = tid; e < CT * CB; e += SCAN_THREADS) {
                    const int i = e / CB, cc = e - i * CB;
                    Vs[i * LV + cc] = i < nt && col0 + cc < p.P ? (col0 + cc < p.Pv ? act_load(v + (size_t)i * p.ldx + cc) : 1.f) : 0.f;
                }
            }
        }
        cp_commit();
    };
    auto stage_sq = [&](float *dst, const float *src, int c) {
        if (c < c1) {
            const float *m = src + ((size_t)c * p.H + h) * CT * CT;
            for (int e = tid; e < CT * (CT / 4); e += SCAN_THREADS) cp16(dst + (e >> 4) * LDC + (e & 15) * 4, m + e * 4, true);
        }
        cp_commit();
    };
    stage_k(c0);
    stage_qv(c0);
    if (DELTA) stage_sq(Ts, p.T, c0);
    else cp_commit();
    stage_sq(Ms, p.M, c0);
    for (int c = c0; c < c1; ++c) {
        const float *Ks = Kb + ((c - c0) & 1) * CT * LD, *F = Fs + ((c - c0) & 1) * FAC;
        const int t0 = p.pieces[2 * c], nt = p.pieces[2 * c + 1] - t0;
        stage_k(c + 1);
        cp_wait<3>();                            // this chunk's K, factors, Q and V
        __syncthreads();
        {
            // half of the threads Q S0, half K S0 (delta) or V's columns as rows
            const int half = tid / (SCAN_THREADS / 2), i0 = tid % (SCAN_THREADS / 2);
            constexpr int TC = CB / 4;
            const Tile<4, TC, 4> tile(i0);
            if (half == 0) {
                float own[4][TC / 4];
                tile.run(Qs, LD, St, LD, D / 4, own);
#pragma unroll
                for (int u = 0; u < TC / 4; ++u)
#pragma unroll
                    for (int q = 0; q < 4; ++q) Ot[tile.col(u) * LDC + tile.row(q)] = F[tile.row(q)] * own[q][u];
            } else if (DELTA) {
                float own[4][TC / 4];
                tile.run(Ks, LD, St, LD, D / 4, own);
#pragma unroll
                for (int u = 0; u < TC / 4; ++u)
#pragma unroll
                    for (int q = 0; q < 4; ++q) {
                        const int i = tile.row(q), cc = tile.col(u);
                        Xt[cc * LDC + i] = fmaf(-F[i], own[q][u], Vs[i * LV + cc]);
                    }
            } else {
                for (int e = i0; e < CT * CB; e += SCAN_THREADS / 2) {
                    const int cc = e >> 6, i = e & 63;
                    const float v = Vs[i * LV + cc];
                    Ut[cc * LDC + i] = v;
                    Wt[cc * LDC + i] = v * F[CT + i];
                }
            }
        }
        cp_wait<2>();                            // T
        __syncthreads();
        stage_qv(c + 1);
        constexpr int RT = CB == 32 ? 4 : 2;
        using Sq = Tile<RT, 4, 4>;
        const Sq sq(tid);
        if (DELTA) {
            float own[RT][1];
            sq.run(Ts, LDC, Xt, LDC, CT / 4, own);
#pragma unroll
            for (int q = 0; q < RT; ++q) {
                const int i = sq.row(q), at = sq.col(0) * LDC + i;
                Ut[at] = own[q][0];
                Wt[at] = own[q][0] * F[CT + i];
            }
        }
        cp_wait<2>();                            // M
        __syncthreads();
        if (DELTA) stage_sq(Ts, p.T, c + 1);
        else cp_commit();
        {
            float own[RT][1];
            sq.run(Ms, LDC, Ut, LDC, CT / 4, own);
#pragma unroll
            for (int q = 0; q < RT; ++q) Ot[sq.col(0) * LDC + sq.row(q)] += own[q][0];      // (the same thread's own element)
        }
        // S = e^(G_last) S + K^T W: a thread has four rows and four columns; with few of them, two or four threads share the tokens
        {
            const int d4 = D / 4, items = d4 * (CB / 4);
            const int parts = 4 * items <= SCAN_THREADS ? 4 : (2 * items <= SCAN_THREADS ? 2 : 1);
            const float eg_last = F[2 * CT];
            for (int it0 = 0; it0 < items; it0 += SCAN_THREADS) {
                const int it = it0 + (parts > 1 ? tid % items : tid), part = parts > 1 ? tid / items : 0;
                const bool on = it < items && part < parts;
                const int dq = it % d4, cq = it / d4;
                float2 acc[4][2];            // [column][two rows]
#pragma unroll
                for (int x = 0; x < 4; ++x) acc[x][0] = acc[x][1] = make_float2(0.f, 0.f);
                if (on) {
                    const int j0 = part * (CT / parts), j1 = j0 + CT / parts;
                    for (int j = j0; j < j1; j += 4) {
                        float4 w4[4];
#pragma unroll
                        for (int x = 0; x < 4; ++x) w4[x] = *reinterpret_cast<const float4 *>(Wt + (cq * 4 + x) * LDC + j);
#pragma unroll
                        for (int y = 0; y < 4; ++y) {
                            const float4 kk = *reinterpret_cast<const float4 *>(Ks + (j + y) * LD + dq * 4);
#pragma unroll
                            for (int x = 0; x < 4; ++x) {
                                const float w = y == 0 ? w4[x].x : y == 1 ? w4[x].y : y == 2 ? w4[x].z : w4[x].w;
                                acc[x][0] = fma2(make_float2(kk.x, kk.y), make_float2(w, w), acc[x][0]);
                                acc[x][1] = fma2(make_float2(kk.z, kk.w), make_float2(w, w), acc[x][1]);
                            }
                        }
                    }
                }
                for (int turn = 0; turn < parts; ++turn) {
                    if (turn > 0) __syncthreads();
                    if (on && part == turn)
#pragma unroll
                        for (int x = 0; x < 4; ++x) {
                            float4 *s = reinterpret_cast<float4 *>(St + (cq * 4 + x) * LD + dq * 4);
                            float4 v = *s;
                            const float f = turn == 0 ? eg_last : 1.f;
                            v.x = fmaf(f, v.x, acc[x][0].x), v.y = fmaf(f, v.y, acc[x][0].y), v.z = fmaf(f, v.z, acc[x][1].x), v.w = fmaf(f, v.w, acc[x][1].y);
                            *s = v;
                        }
                }
            }
        }
        __syncthreads();
        stage_sq(Ms, p.M, c + 1);
        for (int e = tid; e < nt * CB; e += SCAN_THREADS) {
            const int i = e / CB, cc = e - i * CB;
            if (col0 + cc < p.P) p.o[(size_t)(t0 + i) * p.ldo + (size_t)h * p.P + col0 + cc] = Ot[cc * LDC + i];
        }
    }
    cp_wait<0>();
    for (int e = tid; e < D * CB; e += SCAN_THREADS) {
        const int d = p.s_row == 1 ? e % D : e / CB, c = p.s_row == 1 ? e / D : e % CB;
        if (col0 + c < p.P) S_base[(size_t)d * p.s_row + (size_t)(col0 + c) * p.s_col] = St[c * LD + d];
    }
}

size_t scan_floats(int D, int CB, bool delta) {
    return 3 * (size_t)CT * (D + 4) + (delta ? 2 : 1) * (size_t)CT * LDC + (size_t)CT * (CB + 4) + 2 * FAC + (delta ? 4 : 3) * (size_t)CB * LDC +
           (size_t)CB * (D + 4);
}
size_t prep_floats(int D, bool delta) {
    const size_t rows = 2 * (size_t)CT * (D + 4), products = (delta ? 4 : 1) * (size_t)CT * LDC;
    return rows > products ? rows : products;
}
constexpr size_t MAX_SMEM = 227 * 1024;

template <typename K> int allow(K kernel, size_t smem, const char *who) {
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) LGML_FAIL("%s: cannot have %zu bytes of shared memory: %s", who, smem, cudaGetErrorString(e));
    }
    return 0;
}
}  // namespace

// 1 if the chunked form takes keys of D entries (rows of q and k 16-byte aligned: D a multiple of 4)
LGML_API int lgml_chunk_scan_takes(int D, int delta) {
    return D > 0 && D % 4 == 0 && sizeof(float) * scan_floats(D, 16, delta != 0) <= MAX_SMEM && sizeof(float) * prep_floats(D, delta != 0) <= MAX_SMEM - 2048;
}

// q / k: row t of key head g at + t ldx + g D; log_a / w: row t of head h at + t ldg + h lhg; pieces int32 [n_chunks, 2] (first
// token row, the row past the last; at most 64 tokens each).  T (delta) and M float32 [n_chunks, H, 64, 64], fac float32 [n_chunks, H, 132].
LGML_API int lgml_chunk_prepare(const float *q, const float *k, int ldx, const float *log_a, const float *w, int ldg, int lhg, const int *pieces, float *T,
                                float *M, float *fac, int n_chunks, int H, int G, int D, int delta, cudaStream_t stream) {
    LGML_REQUIRE(n_chunks >= 0 && H > 0 && G > 0 && H % G == 0 && G <= 65535 && lgml_chunk_scan_takes(D, delta), "chunk_prepare: bad sizes");
    LGML_REQUIRE(ldx >= G * D && ldx % 4 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)T | (uintptr_t)M | (uintptr_t)fac) & 15) == 0,
                 "chunk_prepare: rows must be 16-byte aligned");
    if (n_chunks == 0) return 0;
    PrepArgs a{q, k, ldx, log_a, w, ldg, lhg, pieces, T, M, fac, H, G, D};
    const size_t smem = sizeof(float) * prep_floats(D, delta != 0);
    dim3 grid(n_chunks, G);
    if (delta) {
        if (allow(chunk_prepare_kernel<true>, smem, "chunk_prepare")) return -1;
        lgml_launch(chunk_prepare_kernel<true>, grid, PREP_THREADS, smem, stream, a);
    } else {
        if (allow(chunk_prepare_kernel<false>, smem, "chunk_prepare")) return -1;
        lgml_launch(chunk_prepare_kernel<false>, grid, PREP_THREADS, smem, stream, a);
    }
    return lgml_launch_status("chunk_prepare");
}

// v: row t of head h at + t ldx + h Pv.  first_piece int32 [n_req + 1], req int32 [n_req] (index into slots).  S(d, col) of head h in a
// slot's row at h D P + d s_row + col s_col.  o: row t of head h at + t ldo + h P.
LGML_API int lgml_chunk_scan(const float *q, const float *k, const float *v, int ldx, const float *T, const float *M, const float *fac, const int *pieces,
                             const int *first_piece, const int *req, float *state, long long state_ld, int s_row, int s_col, const int *slots, float *o,
                             int ldo, int n_req, int H, int G, int D, int Pv, int P, int delta, cudaStream_t stream) {
    LGML_REQUIRE(n_req >= 0 && n_req <= 65535 && H > 0 && H <= 65535 && G > 0 && H % G == 0 && Pv > 0 && P >= Pv && lgml_chunk_scan_takes(D, delta),
                 "chunk_scan: bad sizes");
    LGML_REQUIRE(ldx % 4 == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)T | (uintptr_t)M | (uintptr_t)fac) & 15) == 0, "chunk_scan: rows must be 16-byte aligned");
    LGML_REQUIRE((s_row == 1 && s_col >= D) || (s_col == 1 && s_row >= P), "chunk_scan: the state is neither by rows nor by columns");
    LGML_REQUIRE(state_ld >= (long long)H * D * P && ldo >= H * P, "chunk_scan: rows too short");
    if (n_req == 0) return 0;
    const int v_vec = Pv % 4 == 0 && ((uintptr_t)v & 15) == 0;
    ScanArgs a{q, k, v, ldx, T, M, fac, pieces, first_piece, req, state, state_ld, s_row, s_col, slots, o, ldo, H, G, D, Pv, P, v_vec};
    // 32 columns a block read K, Q, T and M half as often as 16, but only if the blocks still cover the SMs
    const bool wide = sizeof(float) * scan_floats(D, 32, delta != 0) <= MAX_SMEM && (long long)n_req * H * ((P + 31) / 32) >= 120;
    const int CB = wide ? 32 : 16;
    const size_t smem = sizeof(float) * scan_floats(D, CB, delta != 0);
    dim3 grid((P + CB - 1) / CB, H, n_req);
#define LGML_CS(DELTA, CB)                                                            \
    do {                                                                              \
        if (allow(chunk_scan_kernel<DELTA, CB>, smem, "chunk_scan")) return -1;       \
        lgml_launch(chunk_scan_kernel<DELTA, CB>, grid, SCAN_THREADS, smem, stream, a);    \
    } while (0)
    if (delta) { if (wide) LGML_CS(true, 32); else LGML_CS(true, 16); }
    else { if (wide) LGML_CS(false, 32); else LGML_CS(false, 16); }
#undef LGML_CS
    return lgml_launch_status("chunk_scan");
}
