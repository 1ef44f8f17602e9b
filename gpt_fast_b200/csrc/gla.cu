// Gated linear attention: a linear recurrence over key-value products with a decay per key channel.
//
//     z_t = A2 low_t + b                       low_t: the token's `rank` low-rank numbers
//     a_t = sigmoid(z_t)^(1/tau)               per head and key channel, in (0, 1)
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T      per head [d][dv], 32-bit, zero at the start
//     o_t = S_t^T (q_scale q_t)
//     y_t = o_t / sqrt(mean(o_t^2) + eps) * w * silu(gate_t)        per head (gfb_gated_norm, or the decode kernel itself)
//
// Everything behind the projections is 32-bit.  Decays are kept as g = log2 a_t.
//
// gfb_gla         any number of tokens per sequence: the tokens of a sequence are cut into chunks of PC, all chunks run side by
//                 side in three launches (behind one that makes g).  With G_i the sum of g over the chunk's tokens up to i:
//                   1. per chunk:    U = sum_j (k_j 2^(G_end - G_j)) v_j^T and the chunk's decay 2^G_end   (gla_state_kernel)
//                   2. per element:  S before every chunk, S <- 2^G_end S + U; the last S goes to the cache (gla_scan_kernel)
//                   3. per chunk:    o_i = sum_(j<=i) (sum_c q_ic k_jc 2^(G_ic - G_jc)) v_j + (q_i 2^(G_i)) S (gla_out_kernel)
//                 Every power taken has an exponent of at most zero, whatever the decays: sums run within sub-chunks of SUB
//                 tokens (L below), a pair of tokens in two sub-chunks factors through the decay between the later one's
//                 start and the earlier one's end, and a pair within one takes 2^(L_i - L_j) channel by channel.
// gfb_gla_decode  one token per sequence: decay, state update, output, norm and gate in one pass over the state.
#include "common.cuh"

GFB_DEFINE_LAST_ERROR()

__device__ __forceinline__ float ldw(const void* p, int dt, size_t i) {
    return dt == GFB_BF16 ? __bfloat162float(((const __nv_bfloat16*)p)[i]) : ((const float*)p)[i];
}
// log2(sigmoid(z)^(1/tau)) with factor = log2(e) / tau
__device__ __forceinline__ float log2_decay(float z, float factor) {
    return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * factor;
}

// ---------------------------------------------------------------- the decays of a step's tokens ----
// A block takes DEC_TOKENS tokens and 128 channels; a thread owns a channel: its row of A2 against the tokens' low-rank
// numbers, which sit in shared memory [rank][DEC_TOKENS].
constexpr int DEC_TOKENS = 16;

template <typename T>
__global__ void __launch_bounds__(128)
gla_decay_kernel(const T* __restrict__ src, int ld, int low_off, int rank, const T* __restrict__ a2, const void* __restrict__ bias, int b_dt,
                 float factor, float* __restrict__ g, int n_tokens, int C) {
    extern __shared__ __align__(16) float low[];
    gfb_pdl_launch();
    gfb_pdl_wait();
    const int t0 = blockIdx.x * DEC_TOKENS, c = blockIdx.y * 128 + threadIdx.x;
    for (int e = threadIdx.x; e < rank * DEC_TOKENS; e += 128) {
        const int tt = e / rank, r = e - tt * rank;
        low[r * DEC_TOKENS + tt] = t0 + tt < n_tokens ? gfb_to_f32(src[(size_t)(t0 + tt) * ld + low_off + r]) : 0.f;
    }
    __syncthreads();
    if (c >= C) return;
    float acc[DEC_TOKENS];
#pragma unroll
    for (int i = 0; i < DEC_TOKENS; i++) acc[i] = 0.f;
    const T* row = a2 + (size_t)c * rank;
    constexpr int N = 16 / sizeof(T);                // numbers of a row per 16-byte load
    const bool wide = rank % N == 0 && (reinterpret_cast<uintptr_t>(a2) & 15) == 0;
    uint4 raw = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll 8
    for (int r = 0; r < rank; r++) {
        if (wide && r % N == 0) raw = *reinterpret_cast<const uint4*>(row + r);
        const float w = gfb_to_f32(wide ? reinterpret_cast<const T*>(&raw)[r % N] : row[r]);
        const float4* l = reinterpret_cast<const float4*>(low + r * DEC_TOKENS);
#pragma unroll
        for (int i = 0; i < DEC_TOKENS / 4; i++) {
            const float4 v = l[i];
            acc[4 * i] = fmaf(w, v.x, acc[4 * i]); acc[4 * i + 1] = fmaf(w, v.y, acc[4 * i + 1]);
            acc[4 * i + 2] = fmaf(w, v.z, acc[4 * i + 2]); acc[4 * i + 3] = fmaf(w, v.w, acc[4 * i + 3]);
        }
    }
    const float b = ldw(bias, b_dt, c);
#pragma unroll
    for (int i = 0; i < DEC_TOKENS; i++)
        if (t0 + i < n_tokens) g[(size_t)(t0 + i) * C + c] = log2_decay(acc[i] + b, factor);
}

// ---------------------------------------------------------------- chunks side by side ----
constexpr int PC = 64;           // tokens per chunk
constexpr int SUB = 16;          // tokens per sub-chunk
constexpr int THREADS = 256;
// VS below: value columns per block, 64 or (heads that have them) 128; a thread owns VS / 64 groups of four columns, 64 apart

struct ChunkWork { int seq, slot, t0, n; };

// chunks are numbered through the batch, sequence after sequence
__device__ __forceinline__ bool chunk_work(const GfbBatch& b, int w, ChunkWork& c) {
    int left = w;
    for (int i = 0; i < b.n_seqs; i++) {
        const int q0 = b.cu_seqlens[i], qlen = b.cu_seqlens[i + 1] - q0;
        const int nc = (qlen + PC - 1) / PC;
        if (left < nc) {
            c.seq = i;
            c.slot = b.slots[i];
            c.t0 = q0 + left * PC;
            c.n = min(PC, qlen - left * PC);
            return true;
        }
        left -= nc;
    }
    return false;
}

// A block takes 64 key channels and VS value columns.  Thread (channel, sub-chunk) sums the decays of its 16 tokens, then thread
// (ty, tx) owns key channels 4 ty .. + 3 and value columns 4 tx .. + 3 (+ 64) of the product.
template <typename T, int VS>
__global__ void __launch_bounds__(THREADS)
gla_state_kernel(const T* __restrict__ src, int ld, int k_off, int v_off, const float* __restrict__ g, float* __restrict__ U,
                 float* __restrict__ chunk_decay, GfbBatch b, int H, int d, int dv) {
    constexpr int NG = VS / 64;
    extern __shared__ __align__(16) float sm[];
    float* Kc = sm;                                  // [PC][64]: k 2^(the decays behind the token)
    float* Vs = Kc + PC * 64;                        // [PC][VS]
    float* tot = Vs + PC * VS;                       // [4][64]
    gfb_pdl_launch();
    gfb_pdl_wait();
    ChunkWork c;
    if (!chunk_work(b, blockIdx.x, c)) return;
    const int slices = (dv + VS - 1) / VS;
    const int w = blockIdx.x, h = blockIdx.y, v0 = ((int)blockIdx.z % slices) * VS, d0 = ((int)blockIdx.z / slices) * 64;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const int dd = tid & 63, sub = tid >> 6, ch = d0 + dd;
    float gi[SUB], ki[SUB], sum = 0.f;
#pragma unroll
    for (int i = 0; i < SUB; i++) {
        const int j = sub * SUB + i;
        const bool live = j < c.n && ch < d;
        gi[i] = live ? g[(size_t)(c.t0 + j) * H * d + (size_t)h * d + ch] : 0.f;
        ki[i] = live ? gfb_to_f32(src[(size_t)(c.t0 + j) * ld + k_off + h * d + ch]) : 0.f;
    }
#pragma unroll 8
    for (int e = tid; e < PC * VS; e += THREADS) {
        const int j = e / VS, v = e - j * VS;
        Vs[e] = (j < c.n && v0 + v < dv) ? gfb_to_f32(src[(size_t)(c.t0 + j) * ld + v_off + h * dv + v0 + v]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < SUB; i++) sum += gi[i];
    tot[sub * 64 + dd] = sum;
    __syncthreads();
    float after = 0.f;                               // decays behind this sub-chunk
    for (int m = 3; m > sub; m--) after += tot[m * 64 + dd];
    if (v0 == 0 && sub == 0 && ch < d) chunk_decay[((size_t)w * H + h) * d + ch] = exp2f(after + sum);
    float behind = 0.f;                              // decays behind token i within the sub-chunk
#pragma unroll
    for (int i = SUB - 1; i >= 0; i--) {
        Kc[(sub * SUB + i) * 64 + dd] = ki[i] * exp2f(behind + after);
        behind += gi[i];
    }
    __syncthreads();
    float acc[NG][4][4];
#pragma unroll
    for (int n = 0; n < NG; n++)
#pragma unroll
        for (int r = 0; r < 4; r++)
#pragma unroll
            for (int cc = 0; cc < 4; cc++) acc[n][r][cc] = 0.f;
#pragma unroll 4
    for (int j = 0; j < c.n; j++) {
        const float4 k4 = *reinterpret_cast<const float4*>(Kc + j * 64 + 4 * ty);
        const float kk[4] = {k4.x, k4.y, k4.z, k4.w};
#pragma unroll
        for (int n = 0; n < NG; n++) {
            const float4 v4 = *reinterpret_cast<const float4*>(Vs + j * VS + 64 * n + 4 * tx);
            const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
            for (int r = 0; r < 4; r++)
#pragma unroll
                for (int cc = 0; cc < 4; cc++) acc[n][r][cc] = fmaf(kk[r], vv[cc], acc[n][r][cc]);
        }
    }
    float* Ug = U + ((size_t)w * H + h) * d * dv;
    const bool wide = dv % 4 == 0;                    // (U is 16-byte aligned)
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int row = d0 + 4 * ty + r;
        if (row >= d) continue;
#pragma unroll
        for (int n = 0; n < NG; n++) {
            const int v = v0 + 64 * n + 4 * tx;
            if (wide && v < dv) {
                *reinterpret_cast<float4*>(Ug + (size_t)row * dv + v) = make_float4(acc[n][r][0], acc[n][r][1], acc[n][r][2], acc[n][r][3]);
            } else {
#pragma unroll
                for (int cc = 0; cc < 4; cc++)
                    if (v + cc < dv) Ug[(size_t)row * dv + v + cc] = acc[n][r][cc];
            }
        }
    }
}

// a thread per element of a (sequence, head)'s state: U[c] <- S before chunk c, S <- decay_c S + U[c]; the last S is stored
__global__ void __launch_bounds__(256)
gla_scan_kernel(float* __restrict__ U, const float* __restrict__ chunk_decay, float* __restrict__ state, size_t state_ld, GfbBatch b,
                int H, int d, int dv) {
    gfb_pdl_launch();
    gfb_pdl_wait();
    const int s = blockIdx.y, h = blockIdx.z;
    const size_t per = (size_t)d * dv, e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (e >= per) return;
    int first = 0;
    for (int i = 0; i < s; i++) first += (b.cu_seqlens[i + 1] - b.cu_seqlens[i] + PC - 1) / PC;
    const int nc = (b.cu_seqlens[s + 1] - b.cu_seqlens[s] + PC - 1) / PC;
    if (nc == 0) return;
    const int row = (int)(e / dv);
    float* Sg = state + (size_t)b.slots[s] * state_ld + (size_t)h * per + e;
    float S = *Sg;
    // AHEAD chunks' loads are in flight together
    constexpr int AHEAD = 16;
    for (int c = 0; c < nc; c += AHEAD) {
        float add[AHEAD], dec[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; i++) {
            const size_t at = (size_t)(first + min(c + i, nc - 1)) * H + h;
            add[i] = U[at * per + e];
            dec[i] = chunk_decay[at * d + row];
        }
#pragma unroll
        for (int i = 0; i < AHEAD; i++)
            if (c + i < nc) {
                U[((size_t)(first + c + i) * H + h) * per + e] = S;
                S = fmaf(dec[i], S, add[i]);
            }
    }
    *Sg = S;
}

// Thread (ty, tx) of the 16 x 16 grid owns tokens ty + 16 r (one per sub-chunk, r = 0..3) against tokens tx + 16 c, and value
// columns 4 tx .. + 3 (+ 64).  Key channels come DT at a time: q, k and L as they are, qt = q 2^L and kh = k 2^(L_end - L) for pairs in
// different sub-chunks.
constexpr int DT = 32, DTP = DT + 4;
template <int VS>
struct OutSmem {
    union {
        struct { float q[PC][DTP], k[PC][DTP], L[PC][DTP], qt[PC][DTP], kh[PC][DTP]; };
        float A[PC][PC + 4];      // scores, lower triangle (behind the last pass)
    };
    float S[DT][VS];              // the state ahead of the chunk, the channels of this pass
    float V[PC][VS];
    float tot[8][DT];             // decay sums of half sub-chunks
    float M[4][DT];               // decay of a whole sub-chunk
};

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }

template <typename T, int VS>
__global__ void __launch_bounds__(THREADS, 2)
gla_out_kernel(const T* __restrict__ src, int ld, int q_off, int k_off, int v_off, const float* __restrict__ g, const float* __restrict__ U,
               float* __restrict__ out, GfbBatch b, int H, int d, int dv, float q_scale) {
    constexpr int NG = VS / 64;
    extern __shared__ __align__(16) unsigned char raw[];
    OutSmem<VS>& sm = *reinterpret_cast<OutSmem<VS>*>(raw);
    gfb_pdl_launch();
    gfb_pdl_wait();
    ChunkWork c;
    if (!chunk_work(b, blockIdx.x, c)) return;
    const int w = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VS;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    for (int e = tid; e < PC * VS; e += THREADS) {
        const int j = e / VS, v = e - j * VS;
        sm.V[j][v] = (j < c.n && v0 + v < dv) ? gfb_to_f32(src[(size_t)(c.t0 + j) * ld + v_off + h * dv + v0 + v]) : 0.f;
    }
    const float* Ug = U + ((size_t)w * H + h) * d * dv;
    float far[4][4];                                // scores of tokens in different sub-chunks: [r][c], c < r
    float near[4];                                  // scores within a sub-chunk: token ty against tx
    float o[NG][4][4];
#pragma unroll
    for (int r = 0; r < 4; r++) {
        near[r] = 0.f;
#pragma unroll
        for (int cc = 0; cc < 4; cc++) {
            far[r][cc] = 0.f;
#pragma unroll
            for (int n = 0; n < NG; n++) o[n][r][cc] = 0.f;
        }
    }
    const int dd = tid & 31, oct = tid >> 5;        // staging: a channel, eight tokens
    for (int d0 = 0; d0 < d; d0 += DT) {
        const int ch = d0 + dd;
        float gi[8], qi[8], ki[8], sum = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            const int j = oct * 8 + i;
            const bool live = j < c.n && ch < d;
            const T* row = src + (size_t)(c.t0 + (live ? j : 0)) * ld + h * d + (live ? ch : 0);
            sum += live ? g[(size_t)(c.t0 + j) * H * d + (size_t)h * d + ch] : 0.f;
            gi[i] = sum;                             // running sum of the octet
            qi[i] = live ? gfb_to_f32(row[q_off]) * q_scale : 0.f;
            ki[i] = live ? gfb_to_f32(row[k_off]) : 0.f;
        }
        __syncthreads();                            // the previous pass is done with everything below
        sm.tot[oct][dd] = sum;
        for (int e = tid; e < DT * VS; e += THREADS) {
            const int r = e / VS, v = e - r * VS;
            sm.S[r][v] = (d0 + r < d && v0 + v < dv) ? Ug[(size_t)(d0 + r) * dv + v0 + v] : 0.f;
        }
        __syncthreads();
        {
            const float before = (oct & 1) ? sm.tot[oct - 1][dd] : 0.f, whole = sm.tot[oct & ~1][dd] + sm.tot[oct | 1][dd];
            if (!(oct & 1)) sm.M[oct >> 1][dd] = exp2f(whole);
#pragma unroll
            for (int i = 0; i < 8; i++) {
                const int j = oct * 8 + i;
                const float L = gi[i] + before;
                sm.q[j][dd] = qi[i];
                sm.k[j][dd] = ki[i];
                sm.L[j][dd] = L;
                sm.qt[j][dd] = qi[i] * exp2f(L);
                // the decays behind the token within its sub-chunk: never above zero, also where rounding made the two sums cross
                sm.kh[j][dd] = ki[i] * exp2f(fminf(whole - L, 0.f));
            }
        }
        __syncthreads();
#pragma unroll 1
        for (int x = 0; x < DT; x += 4) {
            const float4 M0 = ld4(&sm.M[0][x]), M1 = ld4(&sm.M[1][x]), M2 = ld4(&sm.M[2][x]);
            float4 qt[4];
#pragma unroll
            for (int r = 0; r < 4; r++) qt[r] = ld4(&sm.qt[ty + 16 * r][x]);
            {
                const float4 h0 = ld4(&sm.kh[tx][x]), h1 = ld4(&sm.kh[tx + 16][x]), h2 = ld4(&sm.kh[tx + 32][x]);
                const float4 a2 = make_float4(qt[2].x * M1.x, qt[2].y * M1.y, qt[2].z * M1.z, qt[2].w * M1.w);
                const float4 a3 = make_float4(qt[3].x * M2.x, qt[3].y * M2.y, qt[3].z * M2.z, qt[3].w * M2.w);
                const float4 b3 = make_float4(a3.x * M1.x, a3.y * M1.y, a3.z * M1.z, a3.w * M1.w);
#define DOT4(acc, p, s) acc = fmaf(p.x, s.x, fmaf(p.y, s.y, fmaf(p.z, s.z, fmaf(p.w, s.w, acc))))
                DOT4(far[1][0], qt[1], h0);
                DOT4(far[2][1], qt[2], h1);
                DOT4(far[2][0], a2, h0);
                DOT4(far[3][2], qt[3], h2);
                DOT4(far[3][1], a3, h1);
                DOT4(far[3][0], b3, h0);
#undef DOT4
            }
            if (tx <= ty) {
#pragma unroll
                for (int r = 0; r < 4; r++) {
                    const float4 q4 = ld4(&sm.q[ty + 16 * r][x]), k4 = ld4(&sm.k[tx + 16 * r][x]);
                    const float4 li = ld4(&sm.L[ty + 16 * r][x]), lj = ld4(&sm.L[tx + 16 * r][x]);
                    near[r] = fmaf(q4.x * k4.x, exp2f(li.x - lj.x), near[r]);
                    near[r] = fmaf(q4.y * k4.y, exp2f(li.y - lj.y), near[r]);
                    near[r] = fmaf(q4.z * k4.z, exp2f(li.z - lj.z), near[r]);
                    near[r] = fmaf(q4.w * k4.w, exp2f(li.w - lj.w), near[r]);
                }
            }
            // the carried state: q 2^(L + the sub-chunks before)
            const float p1[4] = {M0.x, M0.y, M0.z, M0.w}, m1[4] = {M1.x, M1.y, M1.z, M1.w}, m2[4] = {M2.x, M2.y, M2.z, M2.w};
#pragma unroll
            for (int y = 0; y < 4; y++) {
                const float p2 = p1[y] * m1[y], p3 = p2 * m2[y];
                const float e[4] = {y == 0 ? qt[0].x : y == 1 ? qt[0].y : y == 2 ? qt[0].z : qt[0].w,
                                    (y == 0 ? qt[1].x : y == 1 ? qt[1].y : y == 2 ? qt[1].z : qt[1].w) * p1[y],
                                    (y == 0 ? qt[2].x : y == 1 ? qt[2].y : y == 2 ? qt[2].z : qt[2].w) * p2,
                                    (y == 0 ? qt[3].x : y == 1 ? qt[3].y : y == 2 ? qt[3].z : qt[3].w) * p3};
#pragma unroll
                for (int n = 0; n < NG; n++) {
                    const float4 s4 = ld4(&sm.S[x + y][64 * n + 4 * tx]);
#pragma unroll
                    for (int r = 0; r < 4; r++) {
                        o[n][r][0] = fmaf(e[r], s4.x, o[n][r][0]); o[n][r][1] = fmaf(e[r], s4.y, o[n][r][1]);
                        o[n][r][2] = fmaf(e[r], s4.z, o[n][r][2]); o[n][r][3] = fmaf(e[r], s4.w, o[n][r][3]);
                    }
                }
            }
        }
    }
    __syncthreads();                                 // the scores take the place of q, k, L
    // scores to shared memory: row ty + 16 r, column tx + 16 c (columns of later sub-chunks are never read)
#pragma unroll
    for (int r = 0; r < 4; r++) {
#pragma unroll
        for (int cc = 0; cc < r; cc++) sm.A[ty + 16 * r][tx + 16 * cc] = far[r][cc];
        sm.A[ty + 16 * r][tx + 16 * r] = tx <= ty ? near[r] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int J = 0; J < 4; J++) {
        if (16 * J >= c.n) break;                    // uniform: no tokens there
#pragma unroll 4
        for (int jj = 0; jj < SUB; jj++) {
            float a[4];
#pragma unroll
            for (int r = J; r < 4; r++) a[r] = sm.A[ty + 16 * r][16 * J + jj];
#pragma unroll
            for (int n = 0; n < NG; n++) {
                const float4 v4 = ld4(&sm.V[16 * J + jj][64 * n + 4 * tx]);
#pragma unroll
                for (int r = J; r < 4; r++) {
                    o[n][r][0] = fmaf(a[r], v4.x, o[n][r][0]); o[n][r][1] = fmaf(a[r], v4.y, o[n][r][1]);
                    o[n][r][2] = fmaf(a[r], v4.z, o[n][r][2]); o[n][r][3] = fmaf(a[r], v4.w, o[n][r][3]);
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < 4; r++) {
        const int i = ty + 16 * r;
        if (i >= c.n) continue;
        float* dst = out + ((size_t)(c.t0 + i) * H + h) * dv;
#pragma unroll
        for (int n = 0; n < NG; n++) {
            const int v = v0 + 64 * n + 4 * tx;
            if (dv % 4 == 0 && v < dv) {              // (out is 16-byte aligned)
                *reinterpret_cast<float4*>(dst + v) = make_float4(o[n][r][0], o[n][r][1], o[n][r][2], o[n][r][3]);
            } else {
#pragma unroll
                for (int cc = 0; cc < 4; cc++)
                    if (v + cc < dv) dst[v + cc] = o[n][r][cc];
            }
        }
    }
}

// Floats of scratch of gfb_gla: the decays of the step's tokens, a state and a decay vector per chunk.
GFB_API long gfb_gla_scratch_floats(int n_tokens, int n_seqs, int H, int d, int dv) {
    const long chunks = (long)n_tokens / PC + n_seqs;
    const long g = ((long)n_tokens * H * d + 3) / 4 * 4, dec = (chunks * H * d + 3) / 4 * 4;
    return g + dec + chunks * H * d * dv;
}

// src [T, ld] of type dt: q (H heads of d) at column q_off, k at k_off, v (H heads of dv) at v_off, the low-rank numbers at low_off;
// a2 [H * d, rank] of type dt, bias [H * d] of b_dt; factor = log2(e) / tau.  state float32, slot stride state_ld, per slot
// [H][d][dv]; out float32 [T, H, dv].
GFB_API int gfb_gla(const void* src, int dt, int ld, int q_off, int k_off, int v_off, int low_off, int rank, const void* a2,
                    const void* bias, int b_dt, float factor, float* state, long state_ld, float* out, float* scratch,
                    const int* cu_seqlens, const int* tok_seq, const int* slots, const int* lengths, int n_seqs, int n_tokens,
                    int H, int d, int dv, float q_scale, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (rank < 1 || H < 1 || d < 1 || dv < 1) return gfb_fail("gfb_gla: rank %d, %d heads of %d and %d", rank, H, d, dv);
    const int chunks = n_tokens / PC + n_seqs;                    // an upper bound; surplus blocks find no work
    const int C = H * d;
    const int vs = dv > 64 ? 128 : 64, slices = (dv + vs - 1) / vs, dtiles = (d + 63) / 64;
    if (H > 65535 || n_seqs > 65535 || (long)slices * dtiles > 65535 || (C + 127) / 128 > 65535)
        return gfb_fail("gfb_gla: %d heads of %d and %d exceed the grid limit", H, d, dv);
    const size_t dsmem = (size_t)rank * DEC_TOKENS * sizeof(float);
    if (dsmem > 48 * 1024) return gfb_fail("gfb_gla: decays of rank %d do not fit shared memory", rank);
    if (((uintptr_t)out | (uintptr_t)scratch) & 15) return gfb_fail("gfb_gla: output and scratch must be 16-byte aligned");
    GfbBatch b{cu_seqlens, tok_seq, slots, lengths, n_seqs, n_tokens};
    float* g = scratch;
    float* decay = g + ((long)n_tokens * C + 3) / 4 * 4;
    float* U = decay + ((long)chunks * C + 3) / 4 * 4;
    const dim3 dgrid((n_tokens + DEC_TOKENS - 1) / DEC_TOKENS, (C + 127) / 128);
    const size_t ssmem = ((size_t)PC * 64 + (size_t)PC * vs + 4 * 64) * sizeof(float);
    cudaError_t e;
#define GO(T, V)                                                                                                                    \
    do {                                                                                                                            \
        static bool configured = false;                                                                                             \
        if (!configured) {                                                                                                          \
            e = cudaFuncSetAttribute(gla_out_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(OutSmem<V>));   \
            if (e == cudaSuccess) e = cudaFuncSetAttribute(gla_state_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ssmem); \
            if (e != cudaSuccess) return gfb_fail("gfb_gla: %s", cudaGetErrorString(e));                                            \
            configured = true;                                                                                                      \
        }                                                                                                                           \
        e = gfb_launch(gla_decay_kernel<T>, dgrid, dim3(128), dsmem, stream, (const T*)src, ld, low_off, rank, (const T*)a2, bias, b_dt, \
                       factor, g, n_tokens, C);                                                                                     \
        if (e == cudaSuccess)                                                                                                       \
            e = gfb_launch(gla_state_kernel<T, V>, dim3(chunks, H, slices * dtiles), dim3(THREADS), ssmem, stream, (const T*)src, ld, k_off, \
                           v_off, (const float*)g, U, decay, b, H, d, dv);                                                          \
        if (e == cudaSuccess)                                                                                                       \
            e = gfb_launch(gla_scan_kernel, dim3((unsigned)(((size_t)d * dv + 255) / 256), n_seqs, H), dim3(256), 0, stream, U,     \
                           (const float*)decay, state, (size_t)state_ld, b, H, d, dv);                                              \
        if (e == cudaSuccess)                                                                                                       \
            e = gfb_launch(gla_out_kernel<T, V>, dim3(chunks, H, slices), dim3(THREADS), sizeof(OutSmem<V>), stream, (const T*)src, ld, q_off, \
                           k_off, v_off, (const float*)g, (const float*)U, out, b, H, d, dv, q_scale);                              \
    } while (0)
    if (dt == GFB_BF16 && vs == 128) GO(__nv_bfloat16, 128);
    else if (dt == GFB_BF16) GO(__nv_bfloat16, 64);
    else if (dt == GFB_F32 && vs == 128) GO(float, 128);
    else if (dt == GFB_F32) GO(float, 64);
    else return gfb_fail("gfb_gla: unknown type %d", dt);
#undef GO
    return gfb_check(e, "gfb_gla");
}

// ---------------------------------------------------------------- one token per sequence ----
// A block per (sequence, head).  Thread (ty, tx) walks over key channels ty, ty + TY, ... with the four value columns 4 tx .. + 3 in
// 16-byte accesses, so the state is read and written once; the partial outputs of a column meet in shared memory and are added
// in ascending order, and the block norms the head and gates it.
constexpr int DEC_THREADS = 512;

template <typename T>
__global__ void __launch_bounds__(DEC_THREADS)
gla_decode_kernel(const T* __restrict__ src, int ld, int q_off, int k_off, int v_off, int low_off, int g_off, int rank,
                  const T* __restrict__ a2, const void* __restrict__ bias, int b_dt, float factor, float* __restrict__ state,
                  size_t state_ld, const void* __restrict__ norm, int n_dt, float eps, T* __restrict__ out, GfbBatch b, int H, int d,
                  int dv, float q_scale) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[32];
    const int txn = dv >> 2, TY = DEC_THREADS / txn;
    float* red = sm;                      // [TY][dv]
    float* qs = red + TY * dv;            // [d]
    float* ks = qs + d;                   // [d]
    float* as = ks + d;                   // [d] decays
    float* low = as + d;                  // [rank]
    gfb_pdl_launch();
    gfb_pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int t = b.cu_seqlens[s];
    const T* row = src + (size_t)t * ld;
    const int tx = tid % txn, ty = tid / txn;
    float4* Sg = reinterpret_cast<float4*>(state + (size_t)b.slots[s] * state_ld + (size_t)h * d * dv) + tx;
    for (int r = tid; r < rank; r += DEC_THREADS) low[r] = gfb_to_f32(row[low_off + r]);
    for (int u = tid; u < d; u += DEC_THREADS) {
        qs[u] = gfb_to_f32(row[q_off + h * d + u]) * q_scale;
        ks[u] = gfb_to_f32(row[k_off + h * d + u]);
    }
    __syncthreads();
    for (int u = tid; u < d; u += DEC_THREADS) {
        const T* ar = a2 + (size_t)(h * d + u) * rank;
        float z = 0.f;
#pragma unroll 8
        for (int r = 0; r < rank; r++) z = fmaf(gfb_to_f32(ar[r]), low[r], z);
        as[u] = exp2f(log2_decay(z + ldw(bias, b_dt, (size_t)h * d + u), factor));
    }
    float vv[4], o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int c = 0; c < 4; c++) vv[c] = ty < TY ? gfb_to_f32(row[v_off + h * dv + 4 * tx + c]) : 0.f;
    __syncthreads();
    if (ty < TY) {
#pragma unroll 8
        for (int u = ty; u < d; u += TY) {
            float4 S4 = Sg[(size_t)u * txn];
            const float a = as[u], k = ks[u], q = qs[u];
            S4.x = fmaf(a, S4.x, k * vv[0]); S4.y = fmaf(a, S4.y, k * vv[1]);
            S4.z = fmaf(a, S4.z, k * vv[2]); S4.w = fmaf(a, S4.w, k * vv[3]);
            Sg[(size_t)u * txn] = S4;
            o[0] = fmaf(S4.x, q, o[0]); o[1] = fmaf(S4.y, q, o[1]); o[2] = fmaf(S4.z, q, o[2]); o[3] = fmaf(S4.w, q, o[3]);
        }
        *reinterpret_cast<float4*>(red + ty * dv + 4 * tx) = make_float4(o[0], o[1], o[2], o[3]);
    }
    __syncthreads();
    float ss = 0.f;
    for (int v = tid; v < dv; v += DEC_THREADS) {
        float acc = 0.f;
        for (int y = 0; y < TY; y++) acc += red[y * dv + v];
        red[v] = acc;                     // a thread reads and writes its own column only
        ss = fmaf(acc, acc, ss);
    }
    ss = gfb_block_sum(ss, scratch);
    const float r = 1.0f / sqrtf(ss / (float)dv + eps);
    for (int v = tid; v < dv; v += DEC_THREADS) {
        const float z = gfb_to_f32(row[g_off + h * dv + v]);
        out[((size_t)t * H + h) * dv + v] = gfb_from_f32<T>(red[v] * r * ldw(norm, n_dt, v) * (z / (1.0f + expf(-z))));
    }
}

// As gfb_gla for steps of one token per sequence, with the gate at column g_off of src and the norm weight [dv] of n_dt; out [T, H * dv]
// of type dt.  Needs dv % 4 == 0, dv <= 2048 and a 16-byte aligned state with state_ld % 4 == 0.
GFB_API int gfb_gla_decode(const void* src, int dt, int ld, int q_off, int k_off, int v_off, int low_off, int g_off, int rank,
                           const void* a2, const void* bias, int b_dt, float factor, float* state, long state_ld, const void* norm,
                           int n_dt, float eps, void* out, const int* cu_seqlens, const int* tok_seq, const int* slots,
                           const int* lengths, int n_seqs, int n_tokens, int H, int d, int dv, float q_scale, cudaStream_t stream) {
    if (n_tokens <= 0 || n_seqs <= 0) return 0;
    if (dv < 4 || dv % 4 || dv > 4 * DEC_THREADS || state_ld % 4 || ((uintptr_t)state & 15))
        return gfb_fail("gfb_gla_decode: value heads of %d or a state stride of %ld do not fit the kernel", dv, state_ld);
    if (rank < 1 || H < 1 || H > 65535 || d < 1) return gfb_fail("gfb_gla_decode: rank %d, %d heads of %d", rank, H, d);
    const size_t smem = ((size_t)(DEC_THREADS / (dv >> 2)) * dv + 3 * (size_t)d + rank) * sizeof(float);
    if (smem > 48 * 1024) return gfb_fail("gfb_gla_decode: %zu bytes of shared memory", smem);
    GfbBatch b{cu_seqlens, tok_seq, slots, lengths, n_seqs, n_tokens};
    cudaError_t e;
    if (dt == GFB_BF16)
        e = gfb_launch(gla_decode_kernel<__nv_bfloat16>, dim3(n_seqs, H), dim3(DEC_THREADS), smem, stream, (const __nv_bfloat16*)src, ld, q_off,
                       k_off, v_off, low_off, g_off, rank, (const __nv_bfloat16*)a2, bias, b_dt, factor, state, (size_t)state_ld, norm, n_dt,
                       eps, (__nv_bfloat16*)out, b, H, d, dv, q_scale);
    else if (dt == GFB_F32)
        e = gfb_launch(gla_decode_kernel<float>, dim3(n_seqs, H), dim3(DEC_THREADS), smem, stream, (const float*)src, ld, q_off, k_off, v_off,
                       low_off, g_off, rank, (const float*)a2, bias, b_dt, factor, state, (size_t)state_ld, norm, n_dt, eps, (float*)out, b,
                       H, d, dv, q_scale);
    else
        return gfb_fail("gfb_gla_decode: unknown type %d", dt);
    return gfb_check(e, "gfb_gla_decode");
}
