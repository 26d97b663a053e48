// The kernel between two blocks whose sub-layers all read the same normed rows: what is pending is brought into the
// residual stream, the row is normed for the next block, and its experts are chosen, in one pass per row.
//
//   x <- x + delta + bias + plus      float, in place (each of the three may be absent)
//   h = x / sqrt(mean(x^2) + eps) * w as act_t
//   z_e = router_e . h, then the experts' weights (router.cuh), all float
//
// delta is the sub-layers' output as act_t, bias a vector that belongs to it (an output projection's), plus float rows that
// join the stream here (the embedding, at the start of a further pass through the same layers).  With a choice of rows
// nothing is written back and nothing is routed: the form before the last norm.
#include "common.cuh"
#include "router.cuh"

#define SNR_THREADS 256
#define SNR_MAX_WIDTH 32768      // the row in shared memory
#define SNR_MAX_SHARED (200 * 1024)

template <typename T, int N> struct alignas(sizeof(T) * N) SnrVec { T v[N]; };

// VEC elements per access (1: any width; 4: widths and bases of that many; the router's rows are then read eight at a
// time where their width allows).  The routing form, which serves a few rows, asks for SNR_BATCH strides of a row before it
// uses the first; the other form serves many rows too and keeps its registers for warps.
#define SNR_BATCH 4
#define SNR_AHEAD 16      // 16-byte loads of a router row that a lane keeps ahead: rows of up to 4,096 bfloat16

template <typename WT, typename RT, int VEC, bool ROUTED>
__global__ void __launch_bounds__(SNR_THREADS) sum_norm_route_kernel(
    float* __restrict__ residual, const act_t* __restrict__ delta, const float* __restrict__ bias,
    const float* __restrict__ plus, const WT* __restrict__ weight, float eps, act_t* __restrict__ out,
    const int* __restrict__ rows, int width, const RT* __restrict__ router, float* __restrict__ shares, const IbRouter R) {
    // the row as float [width], the row that goes out [width], the logits, the router's scratch; each from a multiple of 16 bytes
    extern __shared__ __align__(16) float row_s[];
    act_t* h_s = reinterpret_cast<act_t*>(row_s + (width + 3) / 4 * 4);
    constexpr int BATCH = ROUTED ? SNR_BATCH : 1;
    __shared__ float red[32];
    ib_grid_dependency_launch();
    const int nv = width / VEC;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // weights are written by no kernel: the norm's first stride and each warp's first router row are fetched while the
    // kernel before this one still runs
    SnrVec<WT, VEC> w_first[BATCH];
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
        const int j = threadIdx.x + b * SNR_THREADS;
        if (j < nv) w_first[b] = reinterpret_cast<const SnrVec<WT, VEC>*>(weight)[j];
    }
    constexpr int RV = VEC == 1 ? 1 : 16 / (int)sizeof(RT);           // router elements per load
    const bool wide = VEC > 1 && width % (32 * RV) == 0;               // every lane has the same number of loads
    const int n_logits = R.n_experts + R.has_shared;
    SnrVec<RT, RV> ahead[ROUTED ? SNR_AHEAD : 1];
    const int loads = wide ? width / (32 * RV) : 0;                    // per lane and router row
    const bool kept = ROUTED && wide && loads <= SNR_AHEAD && warp < n_logits;
    auto fetch = [&](int e) {
#pragma unroll
        for (int i = 0; i < (ROUTED ? SNR_AHEAD : 1); ++i)
            if (i < loads) ahead[i] = reinterpret_cast<const SnrVec<RT, RV>*>(router + (long)e * width)[lane + 32 * i];
    };
    if (kept) fetch(warp);
    ib_grid_dependency_wait();
    const long r = rows ? rows[blockIdx.x] : blockIdx.x;
    float* res = residual + r * width;
    const bool write_back = rows == nullptr && (delta || bias || plus);
    float ss = 0.0f;
    for (int j0 = threadIdx.x; j0 < nv; j0 += BATCH * SNR_THREADS) {
        SnrVec<float, VEC> x[BATCH], bs[BATCH], pl[BATCH];
        SnrVec<act_t, VEC> d[BATCH];
#pragma unroll
        for (int b = 0; b < BATCH; ++b) {
            const int j = j0 + b * SNR_THREADS;
            if (j >= nv) break;
            x[b] = reinterpret_cast<const SnrVec<float, VEC>*>(res)[j];
            if (delta) d[b] = reinterpret_cast<const SnrVec<act_t, VEC>*>(delta + r * width)[j];
            if (bias) bs[b] = reinterpret_cast<const SnrVec<float, VEC>*>(bias)[j];
            if (plus) pl[b] = reinterpret_cast<const SnrVec<float, VEC>*>(plus + r * width)[j];
        }
#pragma unroll
        for (int b = 0; b < BATCH; ++b) {
            const int j = j0 + b * SNR_THREADS;
            if (j >= nv) break;
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                if (delta) x[b].v[k] += ib_to_float(d[b].v[k]);
                if (bias) x[b].v[k] += bs[b].v[k];
                if (plus) x[b].v[k] += pl[b].v[k];
                ss += x[b].v[k] * x[b].v[k];
            }
            if (write_back) reinterpret_cast<SnrVec<float, VEC>*>(res)[j] = x[b];
            reinterpret_cast<SnrVec<float, VEC>*>(row_s)[j] = x[b];       // read again by the thread that wrote it
        }
    }
    ss = ib_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
    act_t* dst = out + (long)blockIdx.x * width;
    auto finish = [&](int j, const SnrVec<WT, VEC>& w) {
        const SnrVec<float, VEC> x = reinterpret_cast<const SnrVec<float, VEC>*>(row_s)[j];
        SnrVec<act_t, VEC> o;
#pragma unroll
        for (int k = 0; k < VEC; ++k) o.v[k] = ib_from_float<act_t>(x.v[k] * inv * ib_to_float(w.v[k]));
        reinterpret_cast<SnrVec<act_t, VEC>*>(dst)[j] = o;
        if (ROUTED) reinterpret_cast<SnrVec<act_t, VEC>*>(h_s)[j] = o;
    };
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
        const int j = threadIdx.x + b * SNR_THREADS;
        if (j < nv) finish(j, w_first[b]);
    }
    for (int j = threadIdx.x + BATCH * SNR_THREADS; j < nv; j += SNR_THREADS)
        finish(j, reinterpret_cast<const SnrVec<WT, VEC>*>(weight)[j]);
    if (!ROUTED) return;
    __syncthreads();
    // a warp per expert: the products of the row with the router's rows
    float* logits = row_s + (width + 3) / 4 * 4 + (width * (int)sizeof(act_t) + 15) / 16 * 4;
    for (int e = warp; e < n_logits; e += SNR_THREADS / 32) {
        float dot = 0.0f;
        if (kept) {
#pragma unroll
            for (int i = 0; i < SNR_AHEAD; ++i) {
                if (i >= loads) break;
                const SnrVec<act_t, RV> h = reinterpret_cast<const SnrVec<act_t, RV>*>(h_s)[lane + 32 * i];
#pragma unroll
                for (int k = 0; k < RV; ++k) dot = fmaf(ib_to_float(ahead[ROUTED ? i : 0].v[k]), ib_to_float(h.v[k]), dot);
            }
            if (e + SNR_THREADS / 32 < n_logits) fetch(e + SNR_THREADS / 32);
        } else {
            const SnrVec<RT, VEC>* rw = reinterpret_cast<const SnrVec<RT, VEC>*>(router + (long)e * width);
#pragma unroll 8
            for (int j = lane; j < nv; j += 32) {
                const SnrVec<RT, VEC> a = rw[j];
                const SnrVec<act_t, VEC> h = reinterpret_cast<const SnrVec<act_t, VEC>*>(h_s)[j];
#pragma unroll
                for (int k = 0; k < VEC; ++k) dot = fmaf(ib_to_float(a.v[k]), ib_to_float(h.v[k]), dot);
            }
        }
        dot = ib_warp_sum(dot);
        if (lane == 0) logits[e] = dot;
    }
    __syncthreads();
    if (warp == 0) ib_route_row(logits, logits + (n_logits + 3) / 4 * 4, shares + (long)blockIdx.x * n_logits, R);
}

// residual float [n, width]; delta act_t [n, width], bias float [width], plus float [n, width]: each may be null.  rows
// (or null) chooses n_out rows.  router [n_experts + has_shared, width] (null: nothing is routed), shares
// [n_out, n_experts + has_shared].
IB_EXPORT int ib_sum_norm_route(float* residual, const void* delta, const float* bias, const float* plus,
                                const void* weight, int weight_is_f32, float eps, void* out, const int* rows, int n_out,
                                int width, const void* router, int router_is_f32, float* shares, const float* router_bias,
                                const float* correction, int n_experts, int top, int has_shared, int groups, int keep,
                                int mode, float scale, cudaStream_t stream) {
    if (n_out <= 0) return IB_OK;
    if (width <= 0 || residual == nullptr || weight == nullptr || out == nullptr) return IB_ERR_ARGUMENT;
    if (width > SNR_MAX_WIDTH) return IB_ERR_UNSUPPORTED;
    const IbRouter R = {router_bias, correction, n_experts, top, has_shared ? 1 : 0, mode, groups, keep, scale};
    size_t smem = (size_t)((width + 3) / 4 * 4) * sizeof(float);
    if (router != nullptr) {
        if (!ib_router_ok(R) || shares == nullptr || rows != nullptr) return IB_ERR_ARGUMENT;
        smem += (size_t)((width * (int)sizeof(act_t) + 15) / 16 * 4 + (n_experts + R.has_shared + 3) / 4 * 4 +
                         ib_router_scratch(n_experts)) * sizeof(float);
    }
    if (smem > SNR_MAX_SHARED) return IB_ERR_UNSUPPORTED;
    auto on16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = width % 4 == 0 && on16(residual) && on16(delta) && on16(bias) && on16(plus) && on16(weight) && on16(out) &&
                     on16(router);
#define SNR_LAUNCH(WT, RT, VEC, ROUTED)                                                                               \
    do {                                                                                                              \
        static IbDeviceSet wide;                                                                                      \
        if (smem > 47 * 1024)                                                                                         \
            if (const int e = ib_allow_dynamic_smem(wide, sum_norm_route_kernel<WT, RT, VEC, ROUTED>, SNR_MAX_SHARED)) \
                return e;                                                                                             \
        ib_launch(sum_norm_route_kernel<WT, RT, VEC, ROUTED>, n_out, SNR_THREADS, smem, stream, residual, (const act_t*)delta, \
                  bias, plus, (const WT*)weight, eps, (act_t*)out, rows, width, (const RT*)router, shares, R);         \
    } while (0)
#define SNR_LAUNCH_R(WT, RT) do { if (vec) SNR_LAUNCH(WT, RT, 4, true); else SNR_LAUNCH(WT, RT, 1, true); } while (0)
#define SNR_LAUNCH_N(WT) do { if (vec) SNR_LAUNCH(WT, float, 4, false); else SNR_LAUNCH(WT, float, 1, false); } while (0)
    if (router == nullptr) {
        if (weight_is_f32) SNR_LAUNCH_N(float); else SNR_LAUNCH_N(__nv_bfloat16);
    } else if (weight_is_f32) {
        if (router_is_f32) SNR_LAUNCH_R(float, float); else SNR_LAUNCH_R(float, __nv_bfloat16);
    } else {
        if (router_is_f32) SNR_LAUNCH_R(__nv_bfloat16, float); else SNR_LAUNCH_R(__nv_bfloat16, __nv_bfloat16);
    }
#undef SNR_LAUNCH_N
#undef SNR_LAUNCH_R
#undef SNR_LAUNCH
    return ib_launch_status();
}
