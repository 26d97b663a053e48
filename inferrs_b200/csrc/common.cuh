// Shared helpers of the sm_100a kernels: element types, conversions, reductions, launch checks.
//
// Every library is built twice from the same sources: with -DIB_ACT_BF16=0 the
// activation and cache element `act_t` is float (the true 32-bit path), with
// -DIB_ACT_BF16=1 it is __nv_bfloat16.  Arithmetic inside the kernels is float in
// both builds; only what is stored between kernels changes.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <atomic>

#ifndef IB_ACT_BF16
#error "build with -DIB_ACT_BF16=0 or -DIB_ACT_BF16=1"
#endif

#if IB_ACT_BF16
typedef __nv_bfloat16 act_t;
#else
typedef float act_t;
#endif

#define IB_EXPORT extern "C" __attribute__((visibility("default")))

// Error codes returned by the exported functions.  0 is success; positive values are
// cudaError_t of the launch; negative values are refusals of the arguments.
#define IB_OK 0
#define IB_ERR_UNSUPPORTED (-1)
#define IB_ERR_ARGUMENT (-2)

__device__ __forceinline__ float ib_to_float(float v) { return v; }
__device__ __forceinline__ float ib_to_float(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T ib_from_float(float v);
template <> __device__ __forceinline__ float ib_from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ib_from_float<__nv_bfloat16>(float v) {
    return __float2bfloat16_rn(v);
}

// The first key that a token at position `pos` sees.  span > 0: a sliding window of that many keys
// (pos - span + 1, not below 0); span < 0: chunks of -span positions counted from position 0 of the sequence (the
// first position of pos's own chunk); span == 0: every key from 0 on.
__device__ __forceinline__ int ib_first_visible(int pos, int span) {
    if (span > 0) return pos - span + 1 > 0 ? pos - span + 1 : 0;
    if (span < 0) return pos >= 0 ? (pos / (-span)) * (-span) : 0;
    return 0;
}

// Beside its window a token may also see the first `keep` keys of its sequence (keep 0: it does not).  `lo` is the
// first key of the token's window.
__device__ __forceinline__ bool ib_visible(int j, int lo, int pos, int keep) {
    return j <= pos && (j >= lo || j < keep);
}

// Kernels that walk keys in tiles of `keys` walk the tiles that hold kept keys first and then the window's own, from
// tile t_first on: how many tiles come before t_first, and which tile the i-th one is.
__device__ __forceinline__ int ib_kept_tiles(int keep, int t_first, int keys) {
    const int n = (keep + keys - 1) / keys;
    return n < t_first ? n : t_first;
}
__device__ __forceinline__ int ib_nth_tile(int i, int n_kept, int t_first) {
    return i < n_kept ? i : t_first + i - n_kept;
}

// What the attention kernels may be asked to do beside scale, mask and softmax.  Arrays are [n_heads] or absent.
// head_scale[h] multiplies head h's scaled score; slopes[h] * (pos - j) is taken off it; cap > 0: the score then
// becomes cap * tanh(score / cap); exp(sinks[h]) joins the softmax's denominator once per row (a place without key and
// value, which nothing before it touches).  keep_first: see ib_visible.  gate: head h's output of row r is multiplied
// by sigmoid(gate[r * gate_ld + h]).  A row of the output starts out_ld elements after the row before it.
struct IbScoreOptions {
    const float* head_scale;
    const float* slopes;
    const float* sinks;
    float cap;
    int keep_first;
    const act_t* gate;
    long gate_ld;
    long out_ld;
};

__device__ __forceinline__ float ib_head_gate(const IbScoreOptions& o, long row, int head) {
    return o.gate ? 1.0f / (1.0f + expf(-ib_to_float(o.gate[row * o.gate_ld + head]))) : 1.0f;
}

// The cap for kernels whose scores carry a factor log2(e): with c = cap log2(e), c tanh(x / c) of a score x, through
// tanh(z) = 1 - 2 / (1 + 2^(2 z log2(e))); y is x times ib_cap_factor(cap).  Absolute error about c * 2^-22: far below
// what rounding the keys to bfloat16 does to a score.
static inline float ib_cap_factor(float cap) { return 2.0f / cap; }      // 2 log2(e) / c
__device__ __forceinline__ float ib_capped_log2(float y, float c) {
    float t, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(t) : "f"(y));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.0f + t));         // of infinity: zero
    return fmaf(-2.0f * c, r, c);
}

// 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3)))
__device__ __forceinline__ float ib_gelu_tanh(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

__device__ __forceinline__ float ib_warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

__device__ __forceinline__ float ib_warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Sum over a block of up to 1024 threads; every thread gets the result.  The order of
// the additions depends only on blockDim, so a row's result does not depend on the batch.
__device__ __forceinline__ float ib_block_sum(float v, float* smem32) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = ib_warp_sum(v);
    __syncthreads();  // smem32 may still be read from an earlier call
    if (lane == 0) smem32[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? smem32[lane] : 0.0f;
    r = ib_warp_sum(r);
    return r;
}

// ---------------------------------------------------------------------------------------------
// Programmatic dependent launch.  When the library's switch is on (ib_set_pdl), kernels are launched so
// that they may start before the kernel before them in the stream has finished.  Every kernel of this
// package therefore begins with ib_grid_dependency_sync(): it lets the kernel after it start in turn and
// then waits until the kernel before it has completed and its writes are visible.  Only what no kernel
// writes (weights, tables) may be read before that call.  With the switch off, or for a kernel launched
// the plain way, both instructions do nothing.
// ---------------------------------------------------------------------------------------------
__device__ __forceinline__ void ib_grid_dependency_sync() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
}

// The two halves on their own, for kernels that fetch what no kernel writes (weights, tables, the step's
// description) between them.
__device__ __forceinline__ void ib_grid_dependency_launch() {
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}
__device__ __forceinline__ void ib_grid_dependency_wait() {
    asm volatile("griddepcontrol.wait;" ::: "memory");
}

extern int ib_pdl_enabled;  // one per library, defined beside its exported setter ib_set_pdl

template <typename... KArgs, typename... Args>
static inline void ib_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                             Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ib_pdl_enabled ? 1 : 0;
    cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}

// Dynamic shared memory beyond 48 KB has to be allowed per kernel and per device.  `done` remembers the devices
// of this process on which a kernel has it already (one bit each; a device beyond the 64th is set every time).
// Setting it twice is harmless, so two threads that meet here need no lock.
struct IbDeviceSet { std::atomic<unsigned long long> bits{0}; };

template <typename Kernel>
static inline int ib_allow_dynamic_smem(IbDeviceSet& done, Kernel kernel, size_t bytes) {
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return (int)e;
    const bool tracked = dev >= 0 && dev < 64;
    if (tracked && ((done.bits.load(std::memory_order_acquire) >> dev) & 1ull)) return IB_OK;
    e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
    if (tracked) done.bits.fetch_or(1ull << dev, std::memory_order_release);
    return IB_OK;
}

static inline int ib_launch_status() {
    cudaError_t e = cudaPeekAtLastError();
    return e == cudaSuccess ? IB_OK : (int)e;
}
