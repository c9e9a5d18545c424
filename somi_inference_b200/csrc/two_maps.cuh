// Attention in two maps: a head has two queries and two keys per position, each pair with a softmax
// of its own, over the same values.  With a1 and a2 the outputs of the two maps of a head:
//     d = a1 - factor * a2
//     out = d / sqrt(mean(d^2) + eps) * gain * sigmoid(gate[row, head])          (no gate: 1)
// the mean over the head's value width.  All of it is float32.
//
// Also: which chunks of keys a request reads when some first tokens stay visible beside a window.
#pragma once

#include "common.cuh"

namespace somi {

struct TwoMaps {
    float factor, eps, gain;
    const void* gate;            // logits in the compute dtype, one per row and head; or null
    long long gate_stride;       // elements from row to row
};

// Chunks of `chunk` keys that hold [0, keep) or [first_key, kv_len), numbered first .. end - 1: number
// s is chunk s below n_keep and chunk s + gap from there on.  `compact`: numbered from 0 on without
// those between the kept keys and the window; else (no kept keys) by their place in the sequence.
struct KeptSplits {
    int first, end, n_keep, gap;
};
__device__ __forceinline__ KeptSplits kept_splits(int first_key, int kv_len, int keep, int chunk,
                                                  bool compact) {
    KeptSplits k;
    const int first = first_key / chunk, last = (kv_len + chunk - 1) / chunk;
    if (!compact) {
        k.first = first;
        k.end = last;
        k.n_keep = k.gap = 0;
        return k;
    }
    const int kept = (keep + chunk - 1) / chunk;
    k.first = 0;
    k.n_keep = kept;
    k.gap = first > kept ? first - kept : 0;
    k.end = last - k.gap;
    return k;
}

template <typename T>
__device__ __forceinline__ float two_map_gate(const TwoMaps& two, size_t row, int head) {
    if (two.gate == nullptr) return 1.0f;
    const float z = to_float(static_cast<const T*>(two.gate)[row * two.gate_stride + head]);
    return 1.0f / (1.0f + expf(-z));
}

namespace {      // every file that includes this has kernels of its own (no symbol is shared)

// The merge of split-KV decode attention in two maps: one CTA per (request, head) adds up the
// partial results of both maps and takes their difference.  Warps 0, 2, 4, 6 share the partial
// results of the first map, the others those of the second.  A partial result covers `cpc` chunks.
constexpr int kTwoMergeWarps = 8;
template <int HD>
__global__ void __launch_bounds__(kTwoMergeWarps * 32)
two_map_merge_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, int max_splits,
                     int chunk, int cpc, const int* __restrict__ ctx_len, int row_base, int req_base,
                     int nq, int window, int keep, TwoMaps two, __nv_bfloat16* __restrict__ out) {
    constexpr int V = HD / 32;
    __shared__ float red_o[kTwoMergeWarps][HD];
    __shared__ float red_l[kTwoMergeWarps];
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x, head = blockIdx.y;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, map = warp & 1;
    const int ctx = ctx_len[req_base + i];
    const KeptSplits k = kept_splits(first_visible_key(ctx, window), ctx + 1, keep, chunk, true);
    const int first = k.first / cpc, end = (k.end + cpc - 1) / cpc;
    const size_t base = (static_cast<size_t>(i) * 2 * nq + 2 * head + map) * max_splits;
    float M = -INFINITY;
    for (int s = first + lane; s < end; s += 32) M = fmaxf(M, part_ml[2 * (base + s)]);
    M = warp_max(M);
    float acc[V];
#pragma unroll
    for (int v = 0; v < V; ++v) acc[v] = 0.f;
    float L = 0.f;
#pragma unroll 4
    for (int s = first + (warp >> 1); s < end; s += kTwoMergeWarps / 2) {
        const float2 ml = *reinterpret_cast<const float2*>(part_ml + 2 * (base + s));
        const float f = exp2f(ml.x - M);
        const float* o = part_o + (base + s) * HD;
#pragma unroll
        for (int v = 0; v < V; ++v) acc[v] += f * o[lane + 32 * v];
        L += f * ml.y;
    }
#pragma unroll
    for (int v = 0; v < V; ++v) red_o[warp][lane + 32 * v] = acc[v];
    if (lane == 0) red_l[warp] = L;
    __syncthreads();
    float d = 0.f;
    if (tid < HD) {
        float a[2], l[2];
#pragma unroll
        for (int m = 0; m < 2; ++m) {
            a[m] = l[m] = 0.f;
#pragma unroll
            for (int w = m; w < kTwoMergeWarps; w += 2) {
                a[m] += red_o[w][tid];
                l[m] += red_l[w];
            }
        }
        d = a[0] / l[0] - two.factor * (a[1] / l[1]);
    }
    const float ss = block_sum(d * d, scratch);
    const size_t row = static_cast<size_t>(row_base + i);
    if (tid < HD) {
        const float f = two.gain / sqrtf(ss / static_cast<float>(HD) + two.eps) * two_map_gate<__nv_bfloat16>(two, row, head);
        out[(row * nq + head) * HD + tid] = __float2bfloat16_rn(d * f);
    }
}

}  // namespace

template <int HD>
static int launch_two_map_merge(const float* part_o, const float* part_ml, int max_splits, int chunk,
                                int cpc, const int* ctx_len, int row_base, int req_base, int n_decode,
                                int nq, int window, int keep, const TwoMaps& two, __nv_bfloat16* out,
                                cudaStream_t stream) {
    launch_pdl(two_map_merge_kernel<HD>, dim3(n_decode, nq), dim3(kTwoMergeWarps * 32), 0, stream, part_o,
               part_ml, max_splits, chunk, cpc, ctx_len, row_base, req_base, nq, window, keep, two, out);
    return launch_status();
}

}  // namespace somi
