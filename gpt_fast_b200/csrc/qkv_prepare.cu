// What happens to q, k and v between their projection and the attention, for mixers that the
// rotate-and-append kernel of core.cu does not cover: any subset of
//   - per-head root-mean-square norm of q and of k with a weight shared by the heads
//     (v / sqrt(mean(v^2) + eps) * w, 32-bit), or the same norm over the whole projection
//     (all heads of q, or of k, as one vector, with a weight per column),
//   - rotation of the first rot_dims dimensions of each q and k head by the token's position
//     (pairs (2i, 2i+1) or (i, i + rot_dims/2); the other dimensions pass),
//   - a factor on k,
// and then q to q_out, k and v to the token's place in the paged cache.  Keys and values may have
// different head sizes (dk, dv).  The source row holds q, k and v at given offsets, in the model's
// type or as 32-bit partial sums of a product split over K.
// The per-head norm may come without a weight (NORM_BARE) and may run behind the rotation instead of ahead
// of it (NORM_LAST).  `maps` > 1: every query head and every key head is `maps` vectors of dk side by side
// (several score maps over one set of values); each is normed and rotated as a head of its own, and a cached
// key row holds the `maps` vectors of its head one after the other.
// A projection's biases (one number per column of the source row) are added ahead of everything else.
// One warp per (token, head), the head in shared memory between the steps; with a norm over the whole projection one
// block per token, the token's q, k and v in registers (or, where a rotation pairs numbers of different threads, in shared
// memory) between the steps, so every number is read once.
#include "common.cuh"

GFB_DEFINE_LAST_ERROR()

constexpr int WARPS = 4;
enum { NORM_WHOLE = 1, NORM_BARE = 2, NORM_LAST = 4, Q_SPREAD = 8 };

__device__ __forceinline__ float ld_w(const void* p, int dt, int i) {
    return dt == GFB_BF16 ? __bfloat162float(((const __nv_bfloat16*)p)[i]) : ((const float*)p)[i];
}

template <typename T>
__global__ void __launch_bounds__(WARPS * 32)
qkv_prepare_kernel(const void* __restrict__ src, int S, size_t slice, int width, int q_off, int k_off, int v_off,
                   const void* __restrict__ bias, int b_dt, T* __restrict__ q_out, GfbPagedKV kv, GfbBatch b,
                   const float* __restrict__ table, int table_len, int rot_dims, int pairing, const void* q_norm, const void* k_norm, int w_dt, float eps, float k_scale,
                   int H, int GK, int G, int maps, int dk, int dv, int dmax, int append, int norm_opts, int* status) {
    extern __shared__ float heads[];
    gfb_pdl_launch();
    gfb_pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per_token = H + (append ? GK + G : 0);
    const int norm_whole = norm_opts & NORM_WHOLE;
    const long item = (long)blockIdx.x * WARPS + warp;
    if (item >= (long)b.n_tokens * per_token) return;
    const int t = (int)(item / per_token), head = (int)(item - (long)t * per_token);
    float* v = heads + (size_t)warp * dmax;
    const int s = b.tok_seq[t];
    const int slot = b.slots[s];
    const int pos = b.lengths[slot] + (t - b.cu_seqlens[s]);
    const bool is_q = head < H, is_k = !is_q && head < H + GK;
    const int d = (is_q || is_k) ? dk : dv;
    bool ok = pos >= 0 && (table == nullptr || pos < table_len);
    T* dst = nullptr;
    if (is_q) {
        // Q_SPREAD: q_out rows are maps * dk wide and map m of a head sits at columns m * dk .. of its own row (the rest stays
        // as the caller left it: zeros), so that against a cached row of `maps` keys side by side it meets its own key only
        dst = (norm_opts & Q_SPREAD) ? q_out + (((size_t)t * H + head) * maps + head % maps) * dk : q_out + ((size_t)t * H + head) * dk;
    } else {
        const int pi = pos / kv.page_size, off = pos - pi * kv.page_size;
        const int page = (ok && pi < kv.max_pages) ? kv.page_table[(size_t)slot * kv.max_pages + pi] : -1;
        if (page < 0 || page >= kv.n_pages) ok = false;
        else if (is_k) dst = (T*)kv.k_pool + (((size_t)page * G + (head - H) / maps) * kv.page_size + off) * ((size_t)dk * maps)
                             + (size_t)((head - H) % maps) * dk;
        else dst = (T*)kv.v_pool + (((size_t)page * G + (head - H - GK)) * kv.page_size + off) * dv;
    }
    if (!ok) {
        if (lane == 0 && head == 0) gfb_report(status, GFB_ERR_CACHE_RANGE, t, pos);
        if (is_q) for (int i = lane; i < dk; i += 32) dst[i] = gfb_from_f32<T>(0.f);     // q stays defined
        return;
    }
    const int c0 = is_q ? q_off + head * dk : is_k ? k_off + (head - H) * dk : v_off + (head - H - GK) * dv;
    const size_t e0 = (size_t)t * width + c0;
    float ss = 0.f;
    for (int i = lane; i < d; i += 32) {
        float x;
        if (S > 0) {
            const float* p = (const float*)src;
            x = 0.f;
            for (int k = 0; k < S; k++) x += p[(size_t)k * slice + e0 + i];
        } else {
            x = gfb_to_f32(((const T*)src)[e0 + i]);
        }
        if (bias != nullptr) x += ld_w(bias, b_dt, c0 + i);
        v[i] = x;
        ss += x * x;
    }
    const void* nw = is_q ? q_norm : is_k ? k_norm : nullptr;
    if (nw != nullptr && norm_whole) {
        // the statistic spans every head of the projection; each head's warp adds it up for itself, in the same order
        const int heads = is_q ? H : GK, local = is_q ? head : head - H;
        const size_t p0 = (size_t)t * width + (is_q ? q_off : k_off);
        float tot = 0.f;
        for (int i = lane; i < heads * dk; i += 32) {
            float x;
            if (S > 0) {
                const float* p = (const float*)src;
                x = 0.f;
                for (int k = 0; k < S; k++) x += p[(size_t)k * slice + p0 + i];
            } else {
                x = gfb_to_f32(((const T*)src)[p0 + i]);
            }
            if (bias != nullptr) x += ld_w(bias, b_dt, (is_q ? q_off : k_off) + i);
            tot += x * x;
        }
        tot = gfb_warp_sum(tot);
        const float r = 1.0f / sqrtf(tot / (float)(heads * dk) + eps);
        for (int i = lane; i < d; i += 32) v[i] = v[i] * r * ld_w(nw, w_dt, local * dk + i);
    } else if ((is_q || is_k) && (nw != nullptr || (norm_opts & NORM_BARE)) && !(norm_opts & NORM_LAST)) {
        ss = gfb_warp_sum(ss);
        const float r = 1.0f / sqrtf(ss / (float)d + eps);
        for (int i = lane; i < d; i += 32) v[i] = v[i] * r * (nw != nullptr ? ld_w(nw, w_dt, i) : 1.f);
    }
    __syncwarp();
    const float f = is_k ? k_scale : 1.f;
    if (table != nullptr && (is_q || is_k)) {
        const int half = rot_dims >> 1;
        const float* cs = table + (size_t)pos * half * 2;
        for (int i = lane; i < half; i += 32) {
            const int i0 = pairing == 1 ? i : 2 * i, i1 = pairing == 1 ? i + half : 2 * i + 1;
            const float c = cs[2 * i], sn = cs[2 * i + 1], a = v[i0], bb = v[i1];
            v[i0] = a * c - bb * sn;
            v[i1] = bb * c + a * sn;
        }
        __syncwarp();
    }
    if ((is_q || is_k) && (norm_opts & NORM_LAST) && !norm_whole && (nw != nullptr || (norm_opts & NORM_BARE))) {
        float s2 = 0.f;
        for (int i = lane; i < d; i += 32) s2 += v[i] * v[i];
        s2 = gfb_warp_sum(s2);
        const float r = 1.0f / sqrtf(s2 / (float)d + eps);
        for (int i = lane; i < d; i += 32) v[i] = v[i] * r * (nw != nullptr ? ld_w(nw, w_dt, i) : 1.f);
    }
    for (int i = lane; i < d; i += 32) dst[i] = gfb_from_f32<T>(v[i] * f);
}

// ---- a norm over the whole projection: a block per token -----------------------------------------------
// Shared memory holds the token's q (H heads of dk), k (G of dk) and v (G of dv), biases added.  N = 4: everything moves four
// numbers at a time (columns, head sizes and offsets are multiples of four); N = 1: any sizes.
template <typename T, int N> struct alignas(N * sizeof(T)) AlignedPack { T v[N]; };

template <typename T, int N>
__device__ __forceinline__ float stage_columns(float* dst, const void* __restrict__ src, int S, size_t slice, size_t row, int c0, int n,
                                               const void* __restrict__ bias, int b_dt) {
    float ss = 0.f;
    for (int i = threadIdx.x * N; i < n; i += blockDim.x * N) {
        float x[N];
        if (S > 0) {
            const float* p = (const float*)src + row + c0 + i;
#pragma unroll
            for (int e = 0; e < N; e++) x[e] = 0.f;
            constexpr int W = 4;                                   // partial sums in flight together, added in ascending order
            for (int k = 0; k < S; k += W) {
                AlignedPack<float, N> a[W];
#pragma unroll
                for (int u = 0; u < W; u++) a[u] = *reinterpret_cast<const AlignedPack<float, N>*>(p + (size_t)min(k + u, S - 1) * slice);
#pragma unroll
                for (int u = 0; u < W; u++)
                    if (k + u < S) {
#pragma unroll
                        for (int e = 0; e < N; e++) x[e] += a[u].v[e];
                    }
            }
        } else {
            const AlignedPack<T, N> a = *reinterpret_cast<const AlignedPack<T, N>*>((const T*)src + row + c0 + i);
#pragma unroll
            for (int e = 0; e < N; e++) x[e] = gfb_to_f32(a.v[e]);
        }
#pragma unroll
        for (int e = 0; e < N; e++) {
            if (bias != nullptr) x[e] += ld_w(bias, b_dt, c0 + i + e);
            dst[i + e] = x[e];
            ss += x[e] * x[e];
        }
    }
    return ss;
}

// numbers i .. i + N - 1 of a normed head (v: the head as projected, w0: its first weight), rotated where they lie in the first rot_dims
template <typename T, int N>
__device__ __forceinline__ AlignedPack<T, N> finish_columns(const float* v, int i, float r, const void* w, int w_dt, int w0, const float* cs, int rot_dims,
                                                            int pairing, float f) {
    AlignedPack<T, N> o;
    const int half = rot_dims >> 1;
#pragma unroll
    for (int e = 0; e < N; e++) {
        const int j = i + e;
        float x = v[j] * r * (w != nullptr ? ld_w(w, w_dt, w0 + j) : 1.f);
        if (j < rot_dims) {
            const int pair = pairing == 1 ? (j < half ? j : j - half) : j >> 1;
            const bool first = pairing == 1 ? j < half : !(j & 1);
            const int other = pairing == 1 ? (first ? j + half : j - half) : j ^ 1;
            const float y = v[other] * r * (w != nullptr ? ld_w(w, w_dt, w0 + other) : 1.f);
            const float c = cs[2 * pair], sn = cs[2 * pair + 1];
            x = first ? x * c - y * sn : x * c + y * sn;
        }
        o.v[e] = gfb_from_f32<T>(x * f);
    }
    return o;
}

template <typename T, int N>
__global__ void qkv_prepare_token_kernel(const void* __restrict__ src, int S, size_t slice, int width, int q_off, int k_off, int v_off,
                                         const void* __restrict__ bias, int b_dt, T* __restrict__ q_out, GfbPagedKV kv, GfbBatch b,
                                         const float* __restrict__ table, int table_len, int rot_dims, int pairing, const void* q_norm,
                                         const void* k_norm, int w_dt, float eps, float k_scale, int H, int G, int dk, int dv, int append,
                                         int* status) {
    extern __shared__ __align__(16) float heads[];
    __shared__ float scratch[32];
    gfb_pdl_launch();
    gfb_pdl_wait();
    const int t = blockIdx.x;
    const int s = b.tok_seq[t];
    const int slot = b.slots[s];
    const int pos = b.lengths[slot] + (t - b.cu_seqlens[s]);
    const int nq = H * dk, nk = append ? G * dk : 0, nv = append ? G * dv : 0;
    bool ok = pos >= 0 && (table == nullptr || pos < table_len);
    int page = -1, off = 0;
    if (append && ok) {
        const int pi = pos / kv.page_size;
        off = pos - pi * kv.page_size;
        page = pi < kv.max_pages ? kv.page_table[(size_t)slot * kv.max_pages + pi] : -1;
        ok = page >= 0 && page < kv.n_pages;
    }
    if (!ok) {
        if (threadIdx.x == 0) gfb_report(status, GFB_ERR_CACHE_RANGE, t, pos);
        for (int i = threadIdx.x; i < nq; i += blockDim.x) q_out[(size_t)t * nq + i] = gfb_from_f32<T>(0.f);     // q stays defined
        return;
    }
    const size_t row = (size_t)t * width;
    float* ks = heads + nq;
    float* vs = ks + nk;
    float sq = stage_columns<T, N>(heads, src, S, slice, row, q_off, nq, bias, b_dt);
    float sk = stage_columns<T, N>(ks, src, S, slice, row, k_off, nk, bias, b_dt);
    stage_columns<T, N>(vs, src, S, slice, row, v_off, nv, bias, b_dt);
    sq = gfb_block_sum(sq, scratch);                               // (these also order the staged numbers)
    sk = gfb_block_sum(sk, scratch);
    __syncthreads();
    const float rq = q_norm != nullptr ? 1.0f / sqrtf(sq / (float)nq + eps) : 1.f;
    const float rk = k_norm != nullptr ? 1.0f / sqrtf(sk / (float)max(nk, 1) + eps) : 1.f;
    const float* cs = table != nullptr ? table + (size_t)pos * rot_dims : nullptr;
    for (int i = threadIdx.x * N; i < nq; i += blockDim.x * N) {
        const int h = i / dk, j = i - h * dk;
        *reinterpret_cast<AlignedPack<T, N>*>(q_out + (size_t)t * nq + i) =
            finish_columns<T, N>(heads + h * dk, j, rq, q_norm, w_dt, h * dk, cs, rot_dims, pairing, 1.f);
    }
    for (int i = threadIdx.x * N; i < nk; i += blockDim.x * N) {
        const int g = i / dk, j = i - g * dk;
        T* dst = (T*)kv.k_pool + (((size_t)page * G + g) * kv.page_size + off) * dk + j;
        *reinterpret_cast<AlignedPack<T, N>*>(dst) = finish_columns<T, N>(ks + g * dk, j, rk, k_norm, w_dt, g * dk, cs, rot_dims, pairing, k_scale);
    }
    for (int i = threadIdx.x * N; i < nv; i += blockDim.x * N) {
        const int g = i / dv, j = i - g * dv;
        AlignedPack<T, N> o;
#pragma unroll
        for (int e = 0; e < N; e++) o.v[e] = gfb_from_f32<T>(vs[i + e]);
        *reinterpret_cast<AlignedPack<T, N>*>((T*)kv.v_pool + (((size_t)page * G + g) * kv.page_size + off) * dv + j) = o;
    }
}

// The same with the token's numbers in registers, NP packs of four per thread: for rotations whose pairs are neighbours (or none),
// where nothing a thread needs lies with another one but the two mean squares.  A block takes every gridDim.x-th token; a thread's
// columns, and with them its biases and norm weights, are the same for all of them and are fetched once.
__device__ __forceinline__ void ld_w4(float (&v)[4], const void* p, int dt, int i) {          // i: a multiple of four
    if (dt == GFB_BF16) {
        const AlignedPack<__nv_bfloat16, 4> a = *reinterpret_cast<const AlignedPack<__nv_bfloat16, 4>*>((const __nv_bfloat16*)p + i);
#pragma unroll
        for (int e = 0; e < 4; e++) v[e] = __bfloat162float(a.v[e]);
    } else {
        const float4 a = *reinterpret_cast<const float4*>((const float*)p + i);
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    }
}

constexpr int regs_threads(int np) { return np == 1 ? 1024 : np == 2 ? 768 : 640; }      // the largest block whose registers suffice

template <typename T, int NP>
__global__ void __launch_bounds__(regs_threads(NP)) qkv_prepare_regs_kernel(const void* __restrict__ src, int S, size_t slice, int width, int q_off, int k_off, int v_off,
                                        const void* __restrict__ bias, int b_dt, T* __restrict__ q_out, GfbPagedKV kv, GfbBatch b,
                                        const float* __restrict__ table, int table_len, int rot_dims, const void* q_norm, const void* k_norm,
                                        int w_dt, float eps, float k_scale, int H, int G, int dk, int dv, int append, int* status) {
    __shared__ float2 scratch[2][32];
    const int nq = H * dk, nk = append ? G * dk : 0, nv = append ? G * dv : 0;
    const int cols = nq + nk + nv;
    gfb_pdl_launch();
    // what a pack is, the same for every token: its column in the source row (from), its place in a token's q or, head by head, in
    // its page of keys or values (to), its place in its head (in_head), and its constants
    enum { IS_Q = 0, IS_K = 1, IS_V = 2, NONE = 3 };
    float wt[NP][4], bi[NP][4];
    int kind[NP], from[NP], to[NP], in_head[NP];
#pragma unroll
    for (int p = 0; p < NP; p++) {
        const int i = 4 * (threadIdx.x + p * blockDim.x);
        kind[p] = i < nq ? IS_Q : i < nq + nk ? IS_K : i < cols ? IS_V : NONE;
        from[p] = to[p] = in_head[p] = 0;
#pragma unroll
        for (int e = 0; e < 4; e++) { wt[p][e] = 1.f; bi[p][e] = 0.f; }
        if (kind[p] == NONE) continue;
        const int at = kind[p] == IS_Q ? i : kind[p] == IS_K ? i - nq : i - nq - nk, d = kind[p] == IS_V ? dv : dk;
        const int head = at / d;
        in_head[p] = at - head * d;
        to[p] = kind[p] == IS_Q ? at : head * kv.page_size * d + in_head[p];
        from[p] = (kind[p] == IS_Q ? q_off : kind[p] == IS_K ? k_off : v_off) + at;
        if (kind[p] == IS_Q && q_norm != nullptr) ld_w4(wt[p], q_norm, w_dt, at);
        if (kind[p] == IS_K && k_norm != nullptr) ld_w4(wt[p], k_norm, w_dt, at);
        if (kind[p] == IS_V) in_head[p] = rot_dims;                 // values are not rotated
        if (bias != nullptr) ld_w4(bi[p], bias, b_dt, from[p]);
    }
    gfb_pdl_wait();
    // Where a token goes: a chain of four dependent loads, so one warp looks up the block's next 32 tokens at a time.  What a token
    // brings is fetched while the block still works on the one before it.
    struct Place { int pos, page, off, ok; };
    __shared__ Place places[32];
    auto look_up = [&](int first) {
        const int t = first + (int)threadIdx.x * (int)gridDim.x;
        if (threadIdx.x >= 32 || t >= b.n_tokens) return;
        Place a;
        const int s = b.tok_seq[t];
        const int slot = b.slots[s];
        a.pos = b.lengths[slot] + (t - b.cu_seqlens[s]);
        a.ok = a.pos >= 0 && (table == nullptr || a.pos < table_len);
        a.page = -1;
        a.off = 0;
        if (append && a.ok) {
            const int pi = a.pos / kv.page_size;
            a.off = a.pos - pi * kv.page_size;
            a.page = pi < kv.max_pages ? kv.page_table[(size_t)slot * kv.max_pages + pi] : -1;
            a.ok = a.page >= 0 && a.page < kv.n_pages;
        }
        if (!a.ok) gfb_report(status, GFB_ERR_CACHE_RANGE, t, a.pos);
        places[threadIdx.x] = a;
    };
    AlignedPack<T, 4> raw[NP] = {};                                  // (zeros where there is no pack)
    auto fetch = [&](int t) {
        if (S > 0) return;
        const T* row = (const T*)src + (size_t)t * width;
#pragma unroll
        for (int p = 0; p < NP; p++)
            if (kind[p] != NONE) raw[p] = *reinterpret_cast<const AlignedPack<T, 4>*>(row + from[p]);
    };
    fetch(blockIdx.x);                                               // (a block has at least one token)
    for (int t = blockIdx.x, n = 0; t < b.n_tokens; t += gridDim.x, n = (n + 1) & 31) {
        if (n == 0) {
            if (t != (int)blockIdx.x) __syncthreads();               // everybody has read the last of the earlier 32
            look_up(t);
            __syncthreads();
        }
        float x[NP][4] = {};
        float2 ss = make_float2(0.f, 0.f);                          // q's and k's sums of squares
        if (S > 0) {
#pragma unroll
            for (int p = 0; p < NP; p++) {
                if (kind[p] == NONE) continue;
                const float* f = (const float*)src + (size_t)t * width + from[p];
                float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
                constexpr int W = NP == 1 ? 8 : 4;                  // partial sums in flight together, added in ascending order
                for (int k = 0; k < S; k += W) {
                    float4 a[W];
#pragma unroll
                    for (int u = 0; u < W; u++) a[u] = *reinterpret_cast<const float4*>(f + (size_t)min(k + u, S - 1) * slice);
#pragma unroll
                    for (int u = 0; u < W; u++)
                        if (k + u < S) { v.x += a[u].x; v.y += a[u].y; v.z += a[u].z; v.w += a[u].w; }
                }
                x[p][0] = v.x; x[p][1] = v.y; x[p][2] = v.z; x[p][3] = v.w;
            }
        } else {
#pragma unroll
            for (int p = 0; p < NP; p++)
#pragma unroll
                for (int e = 0; e < 4; e++) x[p][e] = gfb_to_f32(raw[p].v[e]);
        }
        if (t + (int)gridDim.x < b.n_tokens) fetch(t + gridDim.x);
#pragma unroll
        for (int p = 0; p < NP; p++) {
            float sum = 0.f;
#pragma unroll
            for (int e = 0; e < 4; e++) {
                x[p][e] += bi[p][e];
                sum = fmaf(x[p][e], x[p][e], sum);
            }
            ss.x += kind[p] == IS_Q ? sum : 0.f;
            ss.y += kind[p] == IS_K ? sum : 0.f;
        }
        const Place at = places[n];
        {
            // two buffers in turn: a warp may write the next token's sums while another still reads this one's
            const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
            ss.x = gfb_warp_sum(ss.x);
            ss.y = gfb_warp_sum(ss.y);
            if (lane == 0) scratch[n & 1][warp] = ss;
            __syncthreads();
            ss = lane < nwarp ? scratch[n & 1][lane] : make_float2(0.f, 0.f);
            ss.x = gfb_warp_sum(ss.x);
            ss.y = gfb_warp_sum(ss.y);
        }
        const float rq = q_norm != nullptr ? 1.0f / sqrtf(ss.x / (float)nq + eps) : 1.f;
        const float rk = (k_norm != nullptr ? 1.0f / sqrtf(ss.y / (float)max(nk, 1) + eps) : 1.f) * k_scale;
        if (!at.ok) {                                               // the same for every thread of the block
            for (int i = threadIdx.x; i < nq; i += blockDim.x) q_out[(size_t)t * nq + i] = gfb_from_f32<T>(0.f);     // q stays defined
            continue;
        }
        const float* cs = table + (size_t)at.pos * rot_dims;         // (not read where rot_dims is 0)
        T* q_to = q_out + (size_t)t * nq;
        T* k_to = (T*)kv.k_pool + ((size_t)at.page * G * kv.page_size + at.off) * dk;
        T* v_to = (T*)kv.v_pool + ((size_t)at.page * G * kv.page_size + at.off) * dv;
#pragma unroll
        for (int p = 0; p < NP; p++) {
            if (kind[p] == NONE) continue;
            const float r = kind[p] == IS_Q ? rq : kind[p] == IS_K ? rk : 1.f;
#pragma unroll
            for (int e = 0; e < 4; e++) x[p][e] *= r * wt[p][e];
#pragma unroll
            for (int e = 0; e < 4; e += 2)
                if (in_head[p] + e < rot_dims) {
                    const float2 turn = *reinterpret_cast<const float2*>(cs + in_head[p] + e);
                    const float u = x[p][e], v = x[p][e + 1];
                    x[p][e] = u * turn.x - v * turn.y;
                    x[p][e + 1] = v * turn.x + u * turn.y;
                }
            AlignedPack<T, 4> o;
#pragma unroll
            for (int e = 0; e < 4; e++) o.v[e] = gfb_from_f32<T>(x[p][e]);
            *reinterpret_cast<AlignedPack<T, 4>*>((kind[p] == IS_Q ? q_to : kind[p] == IS_K ? k_to : v_to) + to[p]) = o;
        }
    }
}

// how many blocks keep the device full (asked once per kind of kernel and number of threads)
template <typename T, int NP>
static int regs_grid(int threads, int n_tokens) {
    static int resident[33] = {};
    int& r = resident[threads / 32];
    if (r == 0) {
        int per_sm = 0, dev = 0, sms = 0;
        if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per_sm, qkv_prepare_regs_kernel<T, NP>, threads, 0) != cudaSuccess || per_sm < 1) per_sm = 1;
        if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms < 1) sms = 148;
        r = per_sm * sms;
    }
    return n_tokens < r ? n_tokens : r;
}

template <typename T, int N, typename... A>
static cudaError_t launch_token(size_t smem, int n_tokens, int threads, cudaStream_t stream, A... args) {
    if (smem > 40 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(qkv_prepare_token_kernel<T, N>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    return gfb_launch(qkv_prepare_token_kernel<T, N>, dim3((unsigned)n_tokens), dim3((unsigned)threads), smem, stream, args...);
}

// src: [T, width] of type dt, or with n_partials > 0 float32 [n_partials][T][width]; q at q_off (H heads of dk), k at
// k_off (G heads of dk), v at v_off (G heads of dv).  bias (or null): [width] of type b_dt.  table (or null: no rotation): float32 [table_len][rot_dims/2][2].
// q_norm / k_norm (or null): [dk] of type w_dt, or with NORM_WHOLE [H * dk] and [G * dk].  append = 0: only q is produced.
// norm_opts: NORM_WHOLE | NORM_BARE (a per-head norm also where no weight is given) | NORM_LAST (the per-head norm follows
// the rotation) | Q_SPREAD (q_out is [T, H * maps, maps * dk], zeroed by the caller; query j is written at columns
// (j mod maps) * dk of row j).  maps >= 1: H and G count heads; q_out is [T, H * maps, dk], key rows of the cache hold maps * dk numbers.
GFB_API int gfb_qkv_prepare(const void* src, int n_partials, int width, int q_off, int k_off, int v_off, const void* bias, int b_dt,
                            void* q_out, int dt, void* k_pool, void* v_pool, const int* page_table, int max_pages, int page_size, int n_pages,
                            const int* cu_seqlens, const int* tok_seq, const int* slots, const int* lengths, int n_seqs,
                            int n_tokens, const float* table, int table_len, int rot_dims, int pairing,
                            const void* q_norm, const void* k_norm, int w_dt, float eps, float k_scale,
                            int H, int G, int dk, int dv, int append, int norm_opts, int maps, int* status, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (maps < 1) return gfb_fail("gfb_qkv_prepare: %d score maps per head", maps);
    const int HQ = H * maps, GK = G * maps;
    if (table != nullptr && (rot_dims % 2 || rot_dims > dk || rot_dims < 0))
        return gfb_fail("gfb_qkv_prepare: %d rotated dimensions in a head of %d", rot_dims, dk);
    GfbPagedKV kv{k_pool, v_pool, page_table, max_pages, page_size, n_pages};
    GfbBatch b{cu_seqlens, tok_seq, slots, lengths, n_seqs, n_tokens};
    const int dmax = dk > dv ? dk : dv;
    const long items = (long)n_tokens * (HQ + (append ? GK + G : 0));
    const long blocks = (items + WARPS - 1) / WARPS;
    if (blocks > 0x7fffffffL) return gfb_fail("gfb_qkv_prepare: too many heads");
    const size_t smem = (size_t)WARPS * dmax * sizeof(float);
    if (smem > 48 * 1024) return gfb_fail("gfb_qkv_prepare: heads of %d exceed the kernel's shared memory", dmax);
    const size_t slice = (size_t)n_tokens * width;
    cudaError_t e;
    const size_t token_smem = ((size_t)H * dk + (append ? (size_t)G * (dk + dv) : 0)) * sizeof(float);
    if ((norm_opts & NORM_WHOLE) && maps == 1 && !(norm_opts & ~NORM_WHOLE) && token_smem <= 160 * 1024) {
        const bool four = ((q_off | k_off | v_off | width | dk | dv) & 3) == 0
                          && (((uintptr_t)src | (uintptr_t)q_out | (uintptr_t)k_pool | (uintptr_t)v_pool | (uintptr_t)bias | (uintptr_t)q_norm | (uintptr_t)k_norm) & 15) == 0;
        const long cols = (long)H * dk + (append ? (long)G * (dk + dv) : 0);
        if (four && (table == nullptr || pairing == 0)) {
            // few tokens: as many threads as packs (a token's latency is what counts); many: a few packs per thread, several tokens per block
            const int packs = (int)(cols / 4);
            const int most = n_tokens <= 128 ? 1024 : 256;
            const int need = (packs + most - 1) / most;
            const int np = need <= 1 ? 1 : need <= 2 && packs <= 2 * regs_threads(2) ? 2 : 4;
            const int threads = ((packs + np - 1) / np + 31) / 32 * 32;
            if (threads <= regs_threads(np)) {
#define REGS(T, NP) e = gfb_launch(qkv_prepare_regs_kernel<T, NP>, dim3((unsigned)regs_grid<T, NP>(threads, n_tokens)), dim3((unsigned)threads), 0, stream, src, n_partials, slice, width, \
                                   q_off, k_off, v_off, bias, b_dt, (T*)q_out, kv, b, table, table_len, table != nullptr ? rot_dims : 0, q_norm, k_norm, w_dt, eps, \
                                   k_scale, H, G, dk, dv, append, status)
#define REGS_NP(T) do { if (np == 1) REGS(T, 1); else if (np == 2) REGS(T, 2); else REGS(T, 4); } while (0)
                if (dt == GFB_BF16) REGS_NP(__nv_bfloat16);
                else if (dt == GFB_F32) REGS_NP(float);
                else return gfb_fail("gfb_qkv_prepare: unknown type %d", dt);
#undef REGS_NP
#undef REGS
                return gfb_check(e, "gfb_qkv_prepare (registers)");
            }
        }
        const int threads = cols <= 1024 ? 128 : n_tokens <= 128 && cols > 2048 ? 512 : 256;
#define TOKEN(T, N) e = launch_token<T, N>(token_smem, n_tokens, threads, stream, src, n_partials, slice, width, q_off, k_off, v_off, bias, b_dt, \
                                           (T*)q_out, kv, b, table, table_len, table != nullptr ? rot_dims : 0, pairing, q_norm, k_norm, w_dt, eps, k_scale, H, G, \
                                           dk, dv, append, status)
        if (dt == GFB_BF16) { if (four) TOKEN(__nv_bfloat16, 4); else TOKEN(__nv_bfloat16, 1); }
        else if (dt == GFB_F32) { if (four) TOKEN(float, 4); else TOKEN(float, 1); }
        else return gfb_fail("gfb_qkv_prepare: unknown type %d", dt);
#undef TOKEN
        return gfb_check(e, "gfb_qkv_prepare (token)");
    }
#define GO(T) e = gfb_launch(qkv_prepare_kernel<T>, dim3((unsigned)blocks), dim3(WARPS * 32), smem, stream, src, n_partials, slice, \
                             width, q_off, k_off, v_off, bias, b_dt, (T*)q_out, kv, b, table, table_len, rot_dims, pairing, q_norm, k_norm, \
                             w_dt, eps, k_scale, HQ, GK, G, maps, dk, dv, dmax, append, norm_opts, status)
    if (dt == GFB_BF16) GO(__nv_bfloat16);
    else if (dt == GFB_F32) GO(float);
    else return gfb_fail("gfb_qkv_prepare: unknown type %d", dt);
#undef GO
    return gfb_check(e, "gfb_qkv_prepare");
}
