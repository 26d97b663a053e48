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

// VEC elements per access (1: any width; 4: widths and bases of that many)
template <typename WT, typename RT, int VEC>
__global__ void __launch_bounds__(SNR_THREADS) sum_norm_route_kernel(
    float* __restrict__ residual, const act_t* __restrict__ delta, const float* __restrict__ bias,
    const float* __restrict__ plus, const WT* __restrict__ weight, float eps, act_t* __restrict__ out,
    const int* __restrict__ rows, int width, const RT* __restrict__ router, float* __restrict__ shares, const IbRouter R) {
    extern __shared__ __align__(16) float row_s[];      // [width], then [logits], then the router's scratch
    __shared__ float red[32];
    ib_grid_dependency_launch();
    const int nv = width / VEC;
    // the first stride of the weights is fetched while the kernel before this one still runs
    SnrVec<WT, VEC> w_first;
    if ((int)threadIdx.x < nv) w_first = reinterpret_cast<const SnrVec<WT, VEC>*>(weight)[threadIdx.x];
    ib_grid_dependency_wait();
    const long r = rows ? rows[blockIdx.x] : blockIdx.x;
    float* res = residual + r * width;
    const bool write_back = rows == nullptr && (delta || bias || plus);
    float ss = 0.0f;
    for (int j = threadIdx.x; j < nv; j += SNR_THREADS) {
        SnrVec<float, VEC> x = reinterpret_cast<const SnrVec<float, VEC>*>(res)[j];
        if (delta) {
            const SnrVec<act_t, VEC> d = reinterpret_cast<const SnrVec<act_t, VEC>*>(delta + r * width)[j];
#pragma unroll
            for (int k = 0; k < VEC; ++k) x.v[k] += ib_to_float(d.v[k]);
        }
        if (bias) {
            const SnrVec<float, VEC> b = reinterpret_cast<const SnrVec<float, VEC>*>(bias)[j];
#pragma unroll
            for (int k = 0; k < VEC; ++k) x.v[k] += b.v[k];
        }
        if (plus) {
            const SnrVec<float, VEC> p = reinterpret_cast<const SnrVec<float, VEC>*>(plus + r * width)[j];
#pragma unroll
            for (int k = 0; k < VEC; ++k) x.v[k] += p.v[k];
        }
        if (write_back) reinterpret_cast<SnrVec<float, VEC>*>(res)[j] = x;
#pragma unroll
        for (int k = 0; k < VEC; ++k) ss += x.v[k] * x.v[k];
        reinterpret_cast<SnrVec<float, VEC>*>(row_s)[j] = x;       // read again by the thread that wrote it
    }
    ss = ib_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
    act_t* dst = out + (long)blockIdx.x * width;
    for (int j = threadIdx.x; j < nv; j += SNR_THREADS) {
        const SnrVec<float, VEC> x = reinterpret_cast<const SnrVec<float, VEC>*>(row_s)[j];
        const SnrVec<WT, VEC> w = j < SNR_THREADS ? w_first : reinterpret_cast<const SnrVec<WT, VEC>*>(weight)[j];
        SnrVec<act_t, VEC> o;
        SnrVec<float, VEC> h;
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            o.v[k] = ib_from_float<act_t>(x.v[k] * inv * ib_to_float(w.v[k]));
            h.v[k] = ib_to_float(o.v[k]);
        }
        reinterpret_cast<SnrVec<act_t, VEC>*>(dst)[j] = o;
        if (router) reinterpret_cast<SnrVec<float, VEC>*>(row_s)[j] = h;
    }
    if (router == nullptr) return;
    __syncthreads();
    // a warp per expert: the products of the row with the router's rows
    float* logits = row_s + (width + 3) / 4 * 4;
    const int n_logits = R.n_experts + R.has_shared;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int e = warp; e < n_logits; e += SNR_THREADS / 32) {
        const SnrVec<RT, VEC>* rw = reinterpret_cast<const SnrVec<RT, VEC>*>(router + (long)e * width);
        float dot = 0.0f;
#pragma unroll 8
        for (int j = lane; j < nv; j += 32) {
            const SnrVec<RT, VEC> a = rw[j];
            const SnrVec<float, VEC> h = reinterpret_cast<const SnrVec<float, VEC>*>(row_s)[j];
#pragma unroll
            for (int k = 0; k < VEC; ++k) dot = fmaf(ib_to_float(a.v[k]), h.v[k], dot);
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
        smem += (size_t)((n_experts + R.has_shared + 3) / 4 * 4 + ib_router_scratch(n_experts)) * sizeof(float);
    }
    if (smem > SNR_MAX_SHARED) return IB_ERR_UNSUPPORTED;
    auto on16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = width % 4 == 0 && on16(residual) && on16(delta) && on16(bias) && on16(plus) && on16(weight) && on16(out) &&
                     on16(router);
#define SNR_LAUNCH(WT, RT, VEC)                                                                                       \
    do {                                                                                                              \
        static IbDeviceSet wide;                                                                                      \
        if (smem > 47 * 1024)                                                                                         \
            if (const int e = ib_allow_dynamic_smem(wide, sum_norm_route_kernel<WT, RT, VEC>, SNR_MAX_SHARED)) return e; \
        ib_launch(sum_norm_route_kernel<WT, RT, VEC>, n_out, SNR_THREADS, smem, stream, residual, (const act_t*)delta, \
                  bias, plus, (const WT*)weight, eps, (act_t*)out, rows, width, (const RT*)router, shares, R);         \
    } while (0)
#define SNR_LAUNCH_R(WT, RT) do { if (vec) SNR_LAUNCH(WT, RT, 4); else SNR_LAUNCH(WT, RT, 1); } while (0)
    if (weight_is_f32) {
        if (router_is_f32) SNR_LAUNCH_R(float, float); else SNR_LAUNCH_R(float, __nv_bfloat16);
    } else {
        if (router_is_f32) SNR_LAUNCH_R(__nv_bfloat16, float); else SNR_LAUNCH_R(__nv_bfloat16, __nv_bfloat16);
    }
#undef SNR_LAUNCH_R
#undef SNR_LAUNCH
    return ib_launch_status();
}
