// Grouped-query attention over the paged cache, for any head size: one warp per
// (token, query head), 32-bit arithmetic throughout.
//
// A token at position `pos` of its request sees the keys lo..pos of that request,
// lo = 0, pos - window + 1, or (window < 0) the first position of pos's chunk of -window positions.  Values may
// have another size than keys.  This step's keys are already in the cache when the
// kernel runs, so a prompt portion and a decoded token are the same case.  Keys are
// taken 32 at a time in ascending order from a multiple of 32, with an online
// softmax; the order of every sum depends only on (pos, window), never on what else
// is in the batch or on which pages hold the keys.
//
// This is the kernel of the true 32-bit path and the fallback of the bfloat16 path
// for head sizes that its tensor-core kernels do not take.
//
// Two options serve attention whose heads' scores are mixed before the softmax and penalised by distance.
// JOINT: a query head holds one vector per key/value head, side by side (n_kv_heads * head_dim numbers), and its
// score against a token is the sum of its products with all of the token's key heads; values are still those
// of the head's own group.  dist_bias [n_heads, bias_len]: dist_bias[h, pos - j] is taken off head h's score
// against key j (a distance beyond the table reads its last entry).
//
// Three more options, each a number per head (absent: not applied).  head_scale[h] multiplies head h's scaled score
// (a learned temperature).  slopes[h] * (pos - j) is taken off the score (a bias that grows linearly with the
// distance).  sinks[h]: every row's softmax gets one more term, exp(sinks[h]), in its denominator only; no key or
// value belongs to it, and neither the scale nor the factor nor the slope touches it.  The other options (a cap on the
// scores, a sequence's first keys beside the window, a gate per head) are those of IbScoreOptions.
#include "common.cuh"

#define ATT_WARPS 4

template <int DPL, bool JOINT>  // DPL value elements per lane: v_dim <= 32 * DPL
__global__ void paged_attention_generic_kernel(
    const act_t* __restrict__ q, const act_t* __restrict__ k_pages, const act_t* __restrict__ v_pages,
    const int* __restrict__ block_table, int max_pages, int page_size, int n_pages,
    const int* __restrict__ row_request, const int* __restrict__ positions, int n_heads, int n_kv_heads,
    int head_dim, int v_dim, float scale, int window, act_t* __restrict__ out,
    const float* __restrict__ dist_bias, int bias_len, const IbScoreOptions opt) {
    extern __shared__ float smem[];
    ib_grid_dependency_sync();
    const int row = blockIdx.x;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int head = blockIdx.y * ATT_WARPS + warp;
    if (head >= n_heads) return;  // whole warps leave; only warp-level syncs follow
    const int d = head_dim;
    const int dq = JOINT ? n_kv_heads * d : d;      // numbers of a query head
    float* qs = smem + warp * dq;
    const int pos = positions[row];
    const int req = row_request[row];
    const int lo = ib_first_visible(pos, window);
    const int kvh = head / (n_heads / n_kv_heads);
    const int* bt = block_table + (long)req * max_pages;

    const act_t* qr = q + ((long)row * n_heads + head) * dq;
    for (int e = lane; e < dq; e += 32) qs[e] = ib_to_float(qr[e]);
    const float* bias_h = dist_bias ? dist_bias + (long)head * bias_len : nullptr;
    const float scale_h = opt.head_scale ? scale * opt.head_scale[head] : scale;
    const float slope_h = opt.slopes ? opt.slopes[head] : 0.0f;
    __syncwarp();

    float acc[DPL];
#pragma unroll
    for (int k = 0; k < DPL; ++k) acc[k] = 0.0f;
    float m = -INFINITY, l = 0.0f;

    const int n_kept = ib_kept_tiles(opt.keep_first, lo / 32, 32);
    for (int i = 0; ; ++i) {
        const int j0 = ib_nth_tile(i, n_kept, lo / 32) * 32;
        if (j0 > pos) break;
        const int j = j0 + lane;
        const bool valid = ib_visible(j, lo, pos, opt.keep_first);
        float s = -INFINITY;
        long off = 0;      // the key's place counted in heads' rows; times d its key, times v_dim its value
        if (valid) {
            const int page = bt[j / page_size];
            if (page >= 0 && page < n_pages) {
                off = ((long)page * n_kv_heads + kvh) * page_size + (j % page_size);
                float dot = 0.0f;
                if (JOINT) {
                    for (int c = 0; c < n_kv_heads; ++c) {
                        const act_t* kr = k_pages + (((long)page * n_kv_heads + c) * page_size + (j % page_size)) * d;
                        const float* qc = qs + c * d;
                        for (int e = 0; e < d; ++e) dot = fmaf(qc[e], ib_to_float(kr[e]), dot);
                    }
                } else {
                    const act_t* kr = k_pages + off * d;
                    for (int e = 0; e < d; ++e) dot = fmaf(qs[e], ib_to_float(kr[e]), dot);
                }
                s = dot * scale_h - slope_h * (float)(pos - j);
                if (bias_h) s -= bias_h[pos - j < bias_len ? pos - j : bias_len - 1];
                if (opt.cap > 0.0f) s = opt.cap * tanhf(s / opt.cap);
            }
        }
        const float m_new = fmaxf(m, ib_warp_max(s));
        const float p = (s == -INFINITY) ? 0.0f : expf(s - m_new);
        const float corr = (m == -INFINITY) ? 0.0f : expf(m - m_new);
        l = l * corr + ib_warp_sum(p);
#pragma unroll
        for (int k = 0; k < DPL; ++k) acc[k] *= corr;
        const int n_in_chunk = (pos - j0 + 1 < 32) ? pos - j0 + 1 : 32;
        for (int jj = 0; jj < n_in_chunk; ++jj) {
            const float pj = __shfl_sync(0xffffffffu, p, jj);
            const long voff = __shfl_sync(0xffffffffu, off, jj);
            if (pj == 0.0f) continue;  // masked key (uniform over the warp)
            const act_t* vr = v_pages + voff * v_dim;
#pragma unroll
            for (int k = 0; k < DPL; ++k) {
                const int e = lane + 32 * k;
                if (e < v_dim) acc[k] = fmaf(pj, ib_to_float(vr[e]), acc[k]);
            }
        }
        m = m_new;
    }
    if (opt.sinks) {        // the place without a key: it adds to the denominator and to nothing else
        const float sink = opt.sinks[head];
        const float m_new = fmaxf(m, sink);
        const float corr = (m == -INFINITY) ? 0.0f : expf(m - m_new);
        l = l * corr + expf(sink - m_new);
#pragma unroll
        for (int k = 0; k < DPL; ++k) acc[k] *= corr;
    }
    const float inv = (l > 0.0f ? 1.0f / l : 0.0f) * ib_head_gate(opt, row, head);
    act_t* dst = out + row * opt.out_ld + (long)head * v_dim;
#pragma unroll
    for (int k = 0; k < DPL; ++k) {
        const int e = lane + 32 * k;
        if (e < v_dim) dst[e] = ib_from_float<act_t>(acc[k] * inv);
    }
}

IB_EXPORT int ib_paged_attention_generic(const void* q, const void* k_pages, const void* v_pages,
                                         const int* block_table, int max_pages, int page_size, int n_pages,
                                         const int* row_request, const int* positions, int n_rows, int n_heads,
                                         int n_kv_heads, int head_dim, int v_dim, float scale, int window, void* out,
                                         int joint, const float* dist_bias, int bias_len, const float* head_scale,
                                         const float* slopes, const float* sinks, float cap, int keep_first,
                                         const void* gate, long gate_ld, long out_ld, cudaStream_t stream) {
    if (n_rows <= 0) return IB_OK;
    if (n_heads <= 0 || n_kv_heads <= 0 || n_heads % n_kv_heads || head_dim <= 0 || page_size <= 0 || max_pages <= 0)
        return IB_ERR_ARGUMENT;
    if (v_dim <= 0) return IB_ERR_ARGUMENT;
    if (dist_bias != nullptr && bias_len <= 0) return IB_ERR_ARGUMENT;
    if (keep_first < 0 || out_ld < (long)n_heads * v_dim || (gate != nullptr && gate_ld < n_heads)) return IB_ERR_ARGUMENT;
    const IbScoreOptions opt = {head_scale, slopes, sinks, cap, keep_first, (const act_t*)gate, gate_ld, out_ld};
    const int dq = joint ? n_kv_heads * head_dim : head_dim;
    if (head_dim > 512 || v_dim > 512 || dq > 2048) return IB_ERR_UNSUPPORTED;
    const dim3 grid(n_rows, (n_heads + ATT_WARPS - 1) / ATT_WARPS);
    const size_t smem = (size_t)ATT_WARPS * dq * sizeof(float);
#define IB_LAUNCH_ATT_J(DPL, JOINT)                                                                             \
    ib_launch(paged_attention_generic_kernel<DPL, JOINT>, grid, 32 * ATT_WARPS, smem, stream,                   \
        (const act_t*)q, (const act_t*)k_pages, (const act_t*)v_pages, block_table, max_pages, page_size,       \
        n_pages, row_request, positions, n_heads, n_kv_heads, head_dim, v_dim, scale, window, (act_t*)out,      \
        dist_bias, bias_len, opt)
#define IB_LAUNCH_ATT(DPL) do { if (joint) IB_LAUNCH_ATT_J(DPL, true); else IB_LAUNCH_ATT_J(DPL, false); } while (0)
    if (v_dim <= 32) IB_LAUNCH_ATT(1);
    else if (v_dim <= 64) IB_LAUNCH_ATT(2);
    else if (v_dim <= 128) IB_LAUNCH_ATT(4);
    else if (v_dim <= 256) IB_LAUNCH_ATT(8);
    else IB_LAUNCH_ATT(16);
#undef IB_LAUNCH_ATT
#undef IB_LAUNCH_ATT_J
    return ib_launch_status();
}
