// Several residual streams per token instead of one (hyper-connections).
//
// A model keeps NS copies x_1 .. x_NS of the stream (32-bit).  A sublayer reads one weighted sum of them and its output y goes
// back into all of them, which are mixed at the same time:
//
//     (1)  x_t <- sum_s mix[s][t] x_s + leave[t] y          t = 1 .. NS, all from the old streams
//     (2)  u = sum_t enter[t] x_t ;   out = u / sqrt(mean(u^2) + eps) * w      (or u itself, without a norm)
//
// (1) belongs to the sublayer that ends and (2) to the one that begins, and both walk the same columns, so one kernel does both
// in one trip over the row: it reads NS + 1 rows and writes NS rows and the normed one.  y may be one or two addends, each a
// 32-bit tensor or the partial sums [S][T][D] of a product that was split over K (added in ascending order).  The streams of a
// step start out equal: they are then one tensor read NS times (x_stride = 0).  At a step's end (1) is not written back and
// only the rows asked for are computed.
//
// Three forms: a row per block with the row in registers; a row per cluster of blocks for the handful of rows of a decode step;
// any row length and up to MAX_STREAMS streams with the row in shared memory.  Each is one 32-bit sum per number in the same order
// whatever the other rows are.
#include "common.cuh"
#include <cooperative_groups.h>

GFB_DEFINE_LAST_ERROR()

constexpr int MAX_STREAMS = 16;       // of the general form
constexpr int MAX_FAST = 8;           // of the other two, which are built for 1 .. MAX_FAST streams

struct StreamArgs {
    const float* x;          // [NS][T][D], x_stride numbers from stream to stream
    float* x_out;            // where (1) goes, out_stride numbers from stream to stream; null: nowhere
    size_t x_stride, out_stride;
    const float *mix, *leave;            // [NS][NS], [NS]; null: no (1)
    const float *y0, *y1;                // null: none
    int S0, S1;
    size_t slice;
    const float* enter;      // [NS], or null: ones
    const void* w;           // [D] of type w_dt, or null: no norm
    int w_dt;
    float eps;
    void* out;               // [R][D], or null: only (1)
    const int* rows;         // [R], or null
    int NS, D;
};

__device__ __forceinline__ float ld_w(const void* p, int dt, int i) {
    return dt == GFB_BF16 ? __bfloat162float(((const __nv_bfloat16*)p)[i]) : ((const float*)p)[i];
}

__device__ __forceinline__ float4 ld_w4(const void* p, int dt, int i) {          // numbers 4i .. 4i + 3
    if (dt == GFB_BF16) {
        const uint2 raw = reinterpret_cast<const uint2*>(p)[i];
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    return reinterpret_cast<const float4*>(p)[i];
}

__device__ __forceinline__ void fma4(float4& a, float f, const float4& v) {
    a.x = fmaf(f, v.x, a.x); a.y = fmaf(f, v.y, a.y); a.z = fmaf(f, v.z, a.z); a.w = fmaf(f, v.w, a.w);
}

__device__ __forceinline__ void store4(float* o, const float4& v) { *reinterpret_cast<float4*>(o) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* o, const float4& v) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 pk;
    pk.x = *reinterpret_cast<uint32_t*>(&lo);
    pk.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(o) = pk;
}

// the sum of one addend's parts at 4 columns; W loads are in flight together, added in ascending order
template <int W>
__device__ __forceinline__ void add_parts(float4& v, const float* __restrict__ y, int S, size_t slice, size_t at) {
    const float4 first = *reinterpret_cast<const float4*>(y + at);
    v.x += first.x; v.y += first.y; v.z += first.z; v.w += first.w;
    for (int k = 1; k < S; k += W) {
        float4 p[W];
#pragma unroll
        for (int u = 0; u < W; u++) p[u] = *reinterpret_cast<const float4*>(y + (size_t)min(k + u, S - 1) * slice + at);
#pragma unroll
        for (int u = 0; u < W; u++)
            if (k + u < S) { v.x += p[u].x; v.y += p[u].y; v.z += p[u].z; v.w += p[u].w; }
    }
}

// the constants of (1) and (2) into shared memory: mix, then leave, then enter
template <int CAP>
__device__ __forceinline__ void stage_constants(float* c, const StreamArgs& a, int NS) {
    for (int i = threadIdx.x; i < CAP * CAP + 2 * CAP; i += blockDim.x) {
        float v = 0.f;
        if (i < NS * NS) v = a.mix != nullptr ? a.mix[i] : 0.f;
        else if (i >= CAP * CAP && i < CAP * CAP + NS) v = a.leave != nullptr ? a.leave[i - CAP * CAP] : 0.f;
        else if (i >= CAP * CAP + CAP && i < CAP * CAP + CAP + NS) v = a.enter != nullptr ? a.enter[i - CAP * CAP - CAP] : 1.f;
        c[i] = v;
    }
}

// (1) and the weighted sum of (2) at the 4 columns from `col` of row `row`
template <int NS, int W>
__device__ __forceinline__ float4 step4(const StreamArgs& a, const float* __restrict__ c, size_t row, int col) {
    const size_t at = row * a.D + col;
    float4 x[NS];
#pragma unroll
    for (int s = 0; s < NS; s++) x[s] = *reinterpret_cast<const float4*>(a.x + (size_t)s * a.x_stride + at);
    if (a.mix != nullptr) {
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        if (a.y0 != nullptr) add_parts<W>(y, a.y0, a.S0, a.slice, at);
        if (a.y1 != nullptr) add_parts<W>(y, a.y1, a.S1, a.slice, at);
        float4 n[NS];
#pragma unroll
        for (int t = 0; t < NS; t++) {
            n[t] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int s = 0; s < NS; s++) fma4(n[t], c[s * NS + t], x[s]);
            fma4(n[t], c[NS * NS + t], y);
        }
        if (a.x_out != nullptr) {
#pragma unroll
            for (int t = 0; t < NS; t++) *reinterpret_cast<float4*>(a.x_out + (size_t)t * a.out_stride + at) = n[t];
        }
#pragma unroll
        for (int t = 0; t < NS; t++) x[t] = n[t];
    }
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int t = 0; t < NS; t++) fma4(u, c[NS * NS + NS + t], x[t]);
    return u;
}

__device__ __forceinline__ float4 scaled(const float4& u, float r, const float4& g) {
    return make_float4(u.x * r * g.x, u.y * r * g.y, u.z * r * g.z, u.w * r * g.w);
}

// ---------------------------------------------------------------- a row per block, in registers ----
template <typename TO, int NS, int NV>
__global__ void __launch_bounds__(256) streams_row_kernel(StreamArgs a) {
    __shared__ float scratch[32];
    __shared__ float c[NS * NS + 2 * NS];
    gfb_pdl_launch();
    stage_constants<NS>(c, a, NS);
    gfb_pdl_wait();
    __syncthreads();
    const int r = blockIdx.x, nvec = a.D >> 2;
    const size_t row = a.rows != nullptr ? a.rows[r] : r;
    float4 u[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = threadIdx.x + k * blockDim.x;
        u[k] = i < nvec ? step4<NS, 4>(a, c, row, 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        ss += (u[k].x * u[k].x + u[k].y * u[k].y) + (u[k].z * u[k].z + u[k].w * u[k].w);
    }
    if (a.out == nullptr) return;
    float rstd = 1.f;
    if (a.w != nullptr) rstd = 1.0f / sqrtf(gfb_block_sum(ss, scratch) / (float)a.D + a.eps);
#pragma unroll
    for (int k = 0; k < NV; k++) {
        const int i = threadIdx.x + k * blockDim.x;
        if (i >= nvec) continue;
        const float4 g = a.w != nullptr ? ld_w4(a.w, a.w_dt, i) : make_float4(1.f, 1.f, 1.f, 1.f);
        store4((TO*)a.out + (size_t)r * a.D + 4 * i, scaled(u[k], rstd, g));
    }
}

// ---------------------------------------------------------------- a row per cluster of blocks ----
constexpr int ROW_CLUSTER = 8;
constexpr int CLUSTER_THREADS = 128;      // one float4 per thread: rows of up to ROW_CLUSTER * 4 * CLUSTER_THREADS numbers

template <typename TO, int NS>
__global__ void __launch_bounds__(CLUSTER_THREADS) streams_cluster_kernel(StreamArgs a) {
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    __shared__ float scratch[32];
    __shared__ float c[NS * NS + 2 * NS];
    __shared__ float parts[ROW_CLUSTER];                        // every block's sum of squares, pushed here by its owner
    // every block announces that it runs (its shared memory may be written from now on); the matching wait comes just
    // before the first remote write
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    gfb_pdl_launch();
    stage_constants<NS>(c, a, NS);
    const int rank = (int)cluster.block_rank(), chunk = a.D / ROW_CLUSTER, r = blockIdx.y;
    const int col = rank * chunk + 4 * threadIdx.x;
    const bool live = 4 * (int)threadIdx.x < chunk;
    float4 g = make_float4(1.f, 1.f, 1.f, 1.f);                 // weights are no kernel's output: fetched ahead of the wait
    if (live && a.w != nullptr) g = ld_w4(a.w, a.w_dt, col >> 2);
    gfb_pdl_wait();
    __syncthreads();
    const size_t row = a.rows != nullptr ? a.rows[r] : r;
    const float4 u = live ? step4<NS, 8>(a, c, row, col) : make_float4(0.f, 0.f, 0.f, 0.f);
    float ss = (u.x * u.x + u.y * u.y) + (u.z * u.z + u.w * u.w);
    ss = gfb_block_sum(ss, scratch);
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    if (threadIdx.x < ROW_CLUSTER) *cluster.map_shared_rank(&parts[rank], threadIdx.x) = ss;
    cluster.sync();
    float total = 0.f;
#pragma unroll
    for (int k = 0; k < ROW_CLUSTER; k++) total += parts[k];
    const float rstd = a.w != nullptr ? 1.0f / sqrtf(total / (float)a.D + a.eps) : 1.f;
    if (live && a.out != nullptr) store4((TO*)a.out + (size_t)r * a.D + col, scaled(u, rstd, g));
}

// ---------------------------------------------------------------- any row ----
template <typename TO>
__global__ void streams_any_kernel(StreamArgs a) {
    extern __shared__ float u_row[];
    __shared__ float scratch[32];
    __shared__ float c[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
    gfb_pdl_launch();
    const int NS = a.NS;
    stage_constants<MAX_STREAMS>(c, a, NS);
    gfb_pdl_wait();
    __syncthreads();
    const float* leave = c + MAX_STREAMS * MAX_STREAMS;
    const float* enter = leave + MAX_STREAMS;
    const int r = blockIdx.x;
    const size_t base = (size_t)(a.rows != nullptr ? a.rows[r] : r) * a.D;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.D; i += blockDim.x) {
        float x[MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; s++) x[s] = s < NS ? a.x[(size_t)s * a.x_stride + base + i] : 0.f;
        float u = 0.f;
        if (a.mix != nullptr) {
            float y = 0.f;
            if (a.y0 != nullptr) { y += a.y0[base + i]; for (int k = 1; k < a.S0; k++) y += a.y0[(size_t)k * a.slice + base + i]; }
            if (a.y1 != nullptr) { y += a.y1[base + i]; for (int k = 1; k < a.S1; k++) y += a.y1[(size_t)k * a.slice + base + i]; }
            for (int t = 0; t < NS; t++) {
                float n = 0.f;
#pragma unroll
                for (int s = 0; s < MAX_STREAMS; s++)
                    if (s < NS) n = fmaf(c[s * NS + t], x[s], n);
                n = fmaf(leave[t], y, n);
                if (a.x_out != nullptr) a.x_out[(size_t)t * a.out_stride + base + i] = n;
                u = fmaf(enter[t], n, u);
            }
        } else {
#pragma unroll
            for (int s = 0; s < MAX_STREAMS; s++)
                if (s < NS) u = fmaf(enter[s], x[s], u);
        }
        u_row[i] = u;                                            // read back by the same thread only
        ss += u * u;
    }
    if (a.out == nullptr) return;
    float rstd = 1.f;
    if (a.w != nullptr) rstd = 1.0f / sqrtf(gfb_block_sum(ss, scratch) / (float)a.D + a.eps);
    TO* o = (TO*)a.out + (size_t)r * a.D;
    for (int i = threadIdx.x; i < a.D; i += blockDim.x)
        o[i] = gfb_from_f32<TO>(u_row[i] * rstd * (a.w != nullptr ? ld_w(a.w, a.w_dt, i) : 1.f));
}

template <typename TO>
static int launch_streams(const StreamArgs& a, int R, cudaStream_t stream) {
    cudaError_t e;
    const int D = a.D;
    const bool aligned = (((uintptr_t)a.x | (uintptr_t)a.x_out | (uintptr_t)a.y0 | (uintptr_t)a.y1 | (uintptr_t)a.w | (uintptr_t)a.out) & 15) == 0;
    const bool vec = aligned && D % 4 == 0 && a.slice % 4 == 0 && a.x_stride % 4 == 0 && a.out_stride % 4 == 0 && a.NS <= MAX_FAST;
#define BY_NS(GO) switch (a.NS) { case 1: GO(1); break; case 2: GO(2); break; case 3: GO(3); break; case 4: GO(4); break; \
                                  case 5: GO(5); break; case 6: GO(6); break; case 7: GO(7); break; default: GO(8); break; }
    if (vec && R <= 128 && D >= 1024 && D % (4 * ROW_CLUSTER) == 0 && D <= ROW_CLUSTER * 4 * CLUSTER_THREADS) {
#define CGO(N) e = gfb_launch_cluster(streams_cluster_kernel<TO, N>, dim3(ROW_CLUSTER, R), dim3(CLUSTER_THREADS), 0, stream, ROW_CLUSTER, a)
        BY_NS(CGO)
#undef CGO
        return gfb_check(e, "gfb_streams (cluster)");
    }
    const int nvec = D / 4;
    if (vec && nvec <= 8 * 256) {
        const int per = nvec <= 2 * 256 ? 2 : nvec <= 4 * 256 ? 4 : 8;
        int threads = ((nvec + per - 1) / per + 31) / 32 * 32;
#define RGO(N) do { if (per == 2) e = gfb_launch(streams_row_kernel<TO, N, 2>, dim3(R), dim3(threads), 0, stream, a); \
                    else if (per == 4) e = gfb_launch(streams_row_kernel<TO, N, 4>, dim3(R), dim3(threads), 0, stream, a); \
                    else e = gfb_launch(streams_row_kernel<TO, N, 8>, dim3(R), dim3(threads), 0, stream, a); } while (0)
        BY_NS(RGO)
#undef RGO
        return gfb_check(e, "gfb_streams (row)");
    }
#undef BY_NS
    const size_t smem = (size_t)D * sizeof(float);
    if (smem > 200 * 1024) return gfb_fail("gfb_streams: a row of %d elements does not fit shared memory", D);
    if (smem > 40 * 1024) {
        e = cudaFuncSetAttribute(streams_any_kernel<TO>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        if (e != cudaSuccess) return gfb_fail("gfb_streams: %s", cudaGetErrorString(e));
    }
    e = gfb_launch(streams_any_kernel<TO>, dim3(R), dim3(D >= 2048 ? 512 : D >= 512 ? 256 : 128), smem, stream, a);
    return gfb_check(e, "gfb_streams");
}

// x float32 [NS][T][D] (x_stride 0: one row per token that all streams share).  mix [NS][NS] (from, to) and leave [NS], or both null:
// step (1) is left out.  y0 / y1 (or null): float32 [max(S,1)][T][D].  x_out (or null): the new streams; it may be x itself when the
// strides agree.  enter [NS] (or null: ones), w (or null: no norm), out (or null) [R][D] of out_dt.  rows (or null): input rows of
// `out`; nothing is written back then (x_out must be null).
GFB_API int gfb_streams(const float* x, long x_stride, float* x_out, long out_stride, int NS, const float* mix, const float* leave,
                        const float* y0, int S0, const float* y1, int S1, long slice, const float* enter, const void* w, int w_dt,
                        float eps, void* out, int out_dt, const int* rows, int R, int D, cudaStream_t stream) {
    if (R <= 0 || D <= 0) return 0;
    if (NS < 1 || NS > MAX_STREAMS) return gfb_fail("gfb_streams: %d streams (1 to %d)", NS, MAX_STREAMS);
    if ((mix == nullptr) != (leave == nullptr)) return gfb_fail("gfb_streams: the mixing matrix and the output's factors come together");
    if (mix == nullptr && (y0 != nullptr || y1 != nullptr || x_out != nullptr)) return gfb_fail("gfb_streams: a sublayer's output without its constants");
    if (rows != nullptr && x_out != nullptr) return gfb_fail("gfb_streams: a gather of rows writes no streams");
    if (x_out == x && x_out != nullptr && x_stride != out_stride) return gfb_fail("gfb_streams: streams in place keep their stride");
    if (x_out == nullptr && out == nullptr) return 0;
    StreamArgs a{x, x_out, (size_t)x_stride, (size_t)out_stride, mix, leave, y0, y1, S0, S1, (size_t)slice, enter, w, w_dt, eps, out, rows, NS, D};
    if (out == nullptr || out_dt == GFB_F32) return launch_streams<float>(a, R, stream);
    if (out_dt == GFB_BF16) return launch_streams<__nv_bfloat16>(a, R, stream);
    return gfb_fail("gfb_streams: unknown output type %d", out_dt);
}
