// From a row's router logits to a dense row of expert weights, by one warp.  Shared by the router's own kernel and by
// the kernel that norms a row and routes it in one pass.
#pragma once

#include "common.cuh"

// mode 0: the scores are the logits themselves (+ bias), a chosen expert weighs its softmax share among the chosen;
// mode 1: the scores are sigmoid(logits + bias); mode 2: softmax(logits + bias) over all experts; in both a chosen
// expert weighs its score over the sum of the chosen scores (+ 1e-20).  Experts are chosen by score + correction (absent:
// by the score), the `top` largest; equal ones: the lower index.  groups > 0: the experts form that many equal
// groups of neighbours, a group's worth is the sum of its two largest choice scores (its only one in groups of one),
// and only the experts of the `keep` best groups can be chosen.  The weights are multiplied by `scale`.
struct IbRouter {
    const float* bias;         // [n_experts] or null
    const float* correction;   // [n_experts] or null
    int n_experts, top, has_shared, mode, groups, keep;
    float scale;
};

// floats of shared memory that a warp needs
__host__ __device__ inline int ib_router_scratch(int n_experts) { return 5 * n_experts; }

static inline bool ib_router_ok(const IbRouter& R) {
    return R.n_experts > 0 && R.n_experts <= 2048 && R.top > 0 && R.top <= R.n_experts && R.mode >= 0 && R.mode <= 2 &&
           R.groups >= 0 && (R.groups == 0 || (R.n_experts % R.groups == 0 && R.keep > 0 && R.keep <= R.groups &&
                                               (long)R.keep * (R.n_experts / R.groups) >= R.top));
}

// the warp's largest v with its index (the lower one of equals)
__device__ __forceinline__ void ib_warp_argmax(float& v, int& at) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ov > v || (ov == v && oa < at)) { v = ov; at = oa; }
    }
}

// z: the row's logits (n_experts, and one more with has_shared); scratch: ib_router_scratch floats of shared memory of this
// warp's own; weights: the row's n_experts (+ has_shared) results.
__device__ __forceinline__ void ib_route_row(const float* z, float* scratch, float* __restrict__ weights, const IbRouter& R) {
    const int lane = threadIdx.x & 31;
    const int n = R.n_experts;
    constexpr int NONE = 0x7fffffff;
    float* score = scratch;
    float* choice = scratch + n;
    float* taken = scratch + 2 * n;
    float z_max = -INFINITY, z_den = 1.0f;
    if (R.mode == 2) {
        for (int e = lane; e < n; e += 32) z_max = fmaxf(z_max, z[e] + (R.bias ? R.bias[e] : 0.0f));
        z_max = ib_warp_max(z_max);
        float d = 0.0f;
        for (int e = lane; e < n; e += 32) d += expf(z[e] + (R.bias ? R.bias[e] : 0.0f) - z_max);
        z_den = ib_warp_sum(d);
    }
    for (int e = lane; e < n; e += 32) {
        float v = z[e] + (R.bias ? R.bias[e] : 0.0f);
        if (R.mode == 1) v = 1.0f / (1.0f + expf(-v));
        if (R.mode == 2) v = expf(v - z_max) / z_den;
        score[e] = v;
        choice[e] = v + (R.correction ? R.correction[e] : 0.0f);
        taken[e] = 0.0f;
    }
    __syncwarp();
    if (R.groups > 0 && R.keep < R.groups) {
        float* worth = scratch + 3 * n;
        float* kept = scratch + 4 * n;
        const int size = n / R.groups;
        for (int g = lane; g < R.groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;      // the two largest
            for (int e = g * size; e < (g + 1) * size; ++e) {
                const float c = choice[e];
                if (c > a) { b = a; a = c; }
                else if (c > b) b = c;
            }
            worth[g] = size > 1 ? a + b : a;
            kept[g] = 0.0f;
        }
        __syncwarp();
        for (int k = 0; k < R.keep; ++k) {
            float best = -INFINITY;
            int at = NONE;
            for (int g = lane; g < R.groups; g += 32)
                if (kept[g] == 0.0f && (worth[g] > best || (worth[g] == best && g < at))) { best = worth[g]; at = g; }
            ib_warp_argmax(best, at);
            if (at == NONE) break;
            if (lane == 0) kept[at] = 1.0f;
            __syncwarp();
        }
        for (int e = lane; e < n; e += 32)
            if (kept[e / size] == 0.0f) choice[e] = -INFINITY;
        __syncwarp();
    }
    float first = 0.0f, sum = 0.0f;
    for (int k = 0; k < R.top; ++k) {
        float best = -INFINITY;
        int at = NONE;
        for (int e = lane; e < n; e += 32)
            if (taken[e] == 0.0f && choice[e] > best) { best = choice[e]; at = e; }     // ascending e: the lower of equals
        ib_warp_argmax(best, at);
        if (at == NONE) break;        // fewer experts than `top`, or nothing but NaN
        const float s = score[at];
        if (k == 0) first = s;
        sum += R.mode != 0 ? s : expf(s - first);
        __syncwarp();
        if (lane == 0) taken[at] = 1.0f;
        __syncwarp();
    }
    for (int e = lane; e < n; e += 32) {
        float w = 0.0f;
        if (taken[e] != 0.0f) w = (R.mode != 0 ? score[e] / (sum + 1e-20f) : expf(score[e] - first) / sum) * R.scale;
        weights[e] = w;
    }
    if (R.has_shared && lane == 0) weights[n] = 1.0f / (1.0f + expf(-z[n]));
}
