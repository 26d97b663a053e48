// The residual of blocks that norm a sub-layer's input and its output, in one pass per row:
//
//   1. x = source + delta / rms(delta) * post       what the sub-layer before left, through its own norm and scale
//                                                   (no delta: x = source; no post: x = source + delta)
//   2. v = sum_j mix[j] plane_j + mix[J] x          a weighted sum over the J results of earlier layers and x (no mix: v = x)
//   3. out = v / rms(v) * weight                    what the next sub-layer reads
//   4. out = out + c(out)                           a causal convolution over time per channel, in steps in which every
//                                                   request brings one row: the rows before it come from the request's
//                                                   state, which is moved on by one place
//
// x goes to `result` and v to `residual` where they are given.  Everything is float but `delta` and `out`.  The number of
// threads depends on the width alone, so a row's sums do not depend on the step.
#include "common.cuh"

struct SandwichArgs {
    const float* source;
    const act_t* delta;
    const float* post;
    float post_eps;
    const float* planes;        // plane j of row r: planes + j * plane_stride + r * width
    long plane_stride;
    int n_planes;
    const float* mix;           // [n_planes + 1]
    float* result;
    float* residual;
    const void* weight;
    float eps;
    act_t* out;
    const int* rows;            // rows[r] is read for row r of out (source, delta and planes); nothing but out is written
    int width;
    const float* conv_w;        // [taps, width], the last tap weighs the row itself
    int taps;
    float* state;               // [slots, ...], taps - 1 rows of `width` numbers at state_off of a slot, oldest first
    long slot_stride, state_off;
    const int* slots;
    const int* row_request;
};

struct alignas(sizeof(act_t) * 4) SandwichVec4 { act_t v[4]; };

__device__ __forceinline__ void sw_load4(float (&d)[4], const float* p) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    d[0] = t.x; d[1] = t.y; d[2] = t.z; d[3] = t.w;
}
__device__ __forceinline__ void sw_load4(float (&d)[4], const __nv_bfloat16* p) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&t.y));
    d[0] = a.x; d[1] = a.y; d[2] = b.x; d[3] = b.y;
}
__device__ __forceinline__ void sw_store4(float* p, const float (&d)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(d[0], d[1], d[2], d[3]);
}

// The row in registers: NV groups of four columns per thread (thread t has groups t, t + blockDim, ...).  A group
// beyond the row is read as the last one and not written, so that loads carry no condition.
template <typename WT, int NV, int THREADS, bool CONV>
__global__ void __launch_bounds__(THREADS) sandwich_norm_vec_kernel(const SandwichArgs a) {
    __shared__ float red[32];
    ib_grid_dependency_launch();
    const int W = a.width, nv = W >> 2;
    int col[NV];
    bool in[NV];
    float post[NV][4];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int g = threadIdx.x + k * blockDim.x;
        in[k] = g < nv;
        col[k] = min(g, nv - 1) * 4;
        if (a.post) sw_load4(post[k], a.post + col[k]);
        else post[k][0] = post[k][1] = post[k][2] = post[k][3] = 1.0f;
    }
    ib_grid_dependency_wait();
    const int r = blockIdx.x;
    const long src = a.rows ? a.rows[r] : r;
    float x[NV][4], d[NV][4], v[NV][4], cv[CONV ? NV : 1][4];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        sw_load4(x[k], a.source + src * W + col[k]);
        if (a.delta) sw_load4(d[k], a.delta + src * W + col[k]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            v[k][i] = 0.0f;
            if constexpr (CONV) cv[k][i] = 0.0f;
        }
    }
    if (a.mix) {
        const float* p = a.planes + src * W;
#pragma unroll 4
        for (int j = 0; j < a.n_planes; ++j) {
            const float m = a.mix[j];
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                float t[4];
                sw_load4(t, p + (long)j * a.plane_stride + col[k]);
#pragma unroll
                for (int i = 0; i < 4; ++i) v[k][i] = fmaf(m, t[i], v[k][i]);
            }
        }
    }
    float* kept = nullptr;
    if constexpr (CONV) {
        if (a.taps > 1) kept = a.state + (long)a.slots[a.row_request[r]] * a.slot_stride + a.state_off;
        for (int j = 0; j + 1 < a.taps; ++j) {
#pragma unroll
            for (int k = 0; k < NV; ++k) {
                float t[4], w[4];
                sw_load4(t, kept + (long)j * W + col[k]);
                sw_load4(w, a.conv_w + (long)j * W + col[k]);
#pragma unroll
                for (int i = 0; i < 4; ++i) cv[k][i] = fmaf(w[i], t[i], cv[k][i]);
                if (j > 0 && in[k]) sw_store4(kept + (long)(j - 1) * W + col[k], t);
            }
        }
    }
    if (a.delta) {
        float inv = 1.0f;
        if (a.post) {
            float ss = 0.0f;
#pragma unroll
            for (int k = 0; k < NV; ++k)
#pragma unroll
                for (int i = 0; i < 4; ++i) ss = in[k] ? fmaf(d[k][i], d[k][i], ss) : ss;
            ss = ib_block_sum(ss, red);
            inv = 1.0f / sqrtf(ss / (float)W + a.post_eps);
        }
#pragma unroll
        for (int k = 0; k < NV; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) x[k][i] += d[k][i] * inv * post[k][i];
    }
    const float own = a.mix ? a.mix[a.n_planes] : 1.0f;
    float ss = 0.0f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        if (in[k] && a.result) sw_store4(a.result + src * W + col[k], x[k]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            v[k][i] = a.mix ? fmaf(own, x[k][i], v[k][i]) : x[k][i];
            ss = in[k] ? fmaf(v[k][i], v[k][i], ss) : ss;
        }
        if (in[k] && a.residual) sw_store4(a.residual + src * W + col[k], v[k]);
    }
    ss = ib_block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)W + a.eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        float w[4], h[4];
        sw_load4(w, reinterpret_cast<const WT*>(a.weight) + col[k]);
        SandwichVec4 o;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o.v[i] = ib_from_float<act_t>(v[k][i] * inv * w[i]);
            h[i] = ib_to_float(o.v[i]);
        }
        if constexpr (CONV) {
            float cw[4];
            sw_load4(cw, a.conv_w + (long)(a.taps - 1) * W + col[k]);
#pragma unroll
            for (int i = 0; i < 4; ++i) o.v[i] = ib_from_float<act_t>(fmaf(cw[i], h[i], cv[k][i]) + h[i]);
            if (kept && in[k]) sw_store4(kept + (long)(a.taps - 2) * W + col[k], h);
        }
        if (in[k]) *reinterpret_cast<SandwichVec4*>(a.out + (long)r * W + col[k]) = o;
    }
}

// Any width and alignment: the row in shared memory, one number per thread and step.
template <typename WT>
__global__ void sandwich_norm_kernel(const SandwichArgs a) {
    extern __shared__ float sw_row[];
    __shared__ float red[32];
    ib_grid_dependency_sync();
    const int W = a.width, r = blockIdx.x;
    const long src = a.rows ? a.rows[r] : r;
    const act_t* del = a.delta ? a.delta + src * W : nullptr;
    float inv = 1.0f;
    if (del && a.post) {
        float ss = 0.0f;
        for (int j = threadIdx.x; j < W; j += blockDim.x) {
            const float d = ib_to_float(del[j]);
            ss = fmaf(d, d, ss);
        }
        ss = ib_block_sum(ss, red);
        inv = 1.0f / sqrtf(ss / (float)W + a.post_eps);
    }
    float ss = 0.0f;
    for (int j = threadIdx.x; j < W; j += blockDim.x) {
        float x = a.source[src * W + j];
        if (del) x += ib_to_float(del[j]) * inv * (a.post ? a.post[j] : 1.0f);
        if (a.result) a.result[src * W + j] = x;
        if (a.mix) {
            float v = 0.0f;
            for (int p = 0; p < a.n_planes; ++p) v = fmaf(a.mix[p], a.planes[(long)p * a.plane_stride + src * W + j], v);
            x = fmaf(a.mix[a.n_planes], x, v);
        }
        if (a.residual) a.residual[src * W + j] = x;
        sw_row[j] = x;
        ss = fmaf(x, x, ss);
    }
    ss = ib_block_sum(ss, red);
    const float inv_out = 1.0f / sqrtf(ss / (float)W + a.eps);
    float* kept = a.conv_w && a.taps > 1
                      ? a.state + (long)a.slots[a.row_request[r]] * a.slot_stride + a.state_off : nullptr;
    for (int j = threadIdx.x; j < W; j += blockDim.x) {
        act_t o = ib_from_float<act_t>(sw_row[j] * inv_out * ib_to_float(reinterpret_cast<const WT*>(a.weight)[j]));
        if (a.conv_w) {
            const float h = ib_to_float(o);
            float c = 0.0f;
            for (int t = 0; t + 1 < a.taps; ++t) {
                const float k = kept[(long)t * W + j];
                c = fmaf(a.conv_w[(long)t * W + j], k, c);
                if (t > 0) kept[(long)(t - 1) * W + j] = k;
            }
            if (kept) kept[(long)(a.taps - 2) * W + j] = h;
            o = ib_from_float<act_t>(fmaf(a.conv_w[(long)(a.taps - 1) * W + j], h, c) + h);
        }
        a.out[(long)r * W + j] = o;
    }
}

static IbDeviceSet sandwich_smem_f32, sandwich_smem_bf16;

template <typename WT>
static int launch_sandwich(const SandwichArgs& a, int n_rows, bool vec, IbDeviceSet& set, cudaStream_t stream) {
    const int nv = a.width / 4;
    if (vec && nv <= 2048) {
#define IB_SANDWICH(NV, THREADS)                                                                              \
    do {                                                                                                      \
        if (a.conv_w) ib_launch(sandwich_norm_vec_kernel<WT, NV, THREADS, true>, n_rows, THREADS, 0, stream, a); \
        else ib_launch(sandwich_norm_vec_kernel<WT, NV, THREADS, false>, n_rows, THREADS, 0, stream, a);      \
    } while (0)
        if (nv <= 128) IB_SANDWICH(1, 128);
        else if (nv <= 256) IB_SANDWICH(1, 256);
        else if (nv <= 512) IB_SANDWICH(1, 512);
        else if (nv <= 1024) IB_SANDWICH(2, 512);
        else IB_SANDWICH(4, 512);
#undef IB_SANDWICH
        return ib_launch_status();
    }
    const size_t smem = (size_t)a.width * sizeof(float), smem_most = 200 * 1024;
    if (smem > smem_most) return IB_ERR_UNSUPPORTED;
    if (smem > 40 * 1024) {      // (with the static part beside it)
        const int e = ib_allow_dynamic_smem(set, sandwich_norm_kernel<WT>, smem_most);
        if (e != IB_OK) return e;
    }
    ib_launch(sandwich_norm_kernel<WT>, n_rows, a.width >= 512 ? 256 : 128, smem, stream, a);
    return ib_launch_status();
}

// See the head of this file.  delta, post, mix (with planes), result, residual, rows and conv_w may be null; `source`
// and `residual` may be the same tensor.  conv_w asks for one row per request (row r belongs to request
// row_request[r], whose slot is slots[request]) and excludes rows.
IB_EXPORT int ib_sandwich_norm(const float* source, const void* delta, const float* post, float post_eps,
                               const float* planes, long plane_stride, int n_planes, const float* mix, float* result,
                               float* residual, const void* weight, int weight_is_f32, float eps, void* out,
                               const int* rows, int n_rows, int width, const float* conv_w, int taps, float* state,
                               long slot_stride, long state_off, const int* slots, const int* row_request,
                               cudaStream_t stream) {
    if (n_rows <= 0) return IB_OK;
    if (width <= 0 || source == nullptr || weight == nullptr || out == nullptr || n_planes < 0 ||
        (mix != nullptr && n_planes > 0 && planes == nullptr) ||
        (rows != nullptr && (result != nullptr || residual != nullptr || conv_w != nullptr)))
        return IB_ERR_ARGUMENT;
    if (conv_w != nullptr && (taps <= 0 || (taps > 1 && (state == nullptr || slots == nullptr || row_request == nullptr ||
                                                         slot_stride < state_off + (long)(taps - 1) * width))))
        return IB_ERR_ARGUMENT;
    const SandwichArgs a = {source, (const act_t*)delta, post, post_eps, planes, plane_stride, n_planes, mix, result,
                            residual, weight, eps, (act_t*)out, rows, width, conv_w, taps, state, slot_stride, state_off,
                            slots, row_request};
    const uintptr_t ptrs = (uintptr_t)source | (uintptr_t)delta | (uintptr_t)post | (uintptr_t)planes | (uintptr_t)result |
                           (uintptr_t)residual | (uintptr_t)weight | (uintptr_t)out | (uintptr_t)conv_w | (uintptr_t)state;
    const bool vec = (width & 3) == 0 && (ptrs & 15) == 0 && (plane_stride & 3) == 0 && (slot_stride & 3) == 0 &&
                     (state_off & 3) == 0;
    return weight_is_f32 ? launch_sandwich<float>(a, n_rows, vec, sandwich_smem_f32, stream)
                         : launch_sandwich<__nv_bfloat16>(a, n_rows, vec, sandwich_smem_bf16, stream);
}
