// The end of attention in two maps (two_maps.cuh) where the attention kernel has left both maps'
// outputs in memory: float32 rows [T, 2 heads, vd], a head's first map in front of its second.
// One warp per (row, head).
#include "two_maps.cuh"

namespace somi {

template <typename T>
__global__ void two_map_difference_kernel(const float* __restrict__ maps, TwoMaps two, int heads, int vd,
                                          long long n, T* __restrict__ out) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    for (long long it = static_cast<long long>(blockIdx.x) * warps + (threadIdx.x >> 5); it < n;
         it += static_cast<long long>(gridDim.x) * warps) {
        const float* a = maps + it * 2 * vd;
        float ss = 0.f;
        for (int e = lane; e < vd; e += 32) {
            const float d = a[e] - two.factor * a[vd + e];
            ss = fmaf(d, d, ss);
        }
        ss = warp_sum(ss);
        const long long row = it / heads;
        const float f = two.gain / sqrtf(ss / static_cast<float>(vd) + two.eps) *
                        two_map_gate<T>(two, static_cast<size_t>(row), static_cast<int>(it - row * heads));
        for (int e = lane; e < vd; e += 32) out[it * vd + e] = from_float<T>((a[e] - two.factor * a[vd + e]) * f);
    }
}

}  // namespace somi

using namespace somi;

// maps: float32 [rows, 2 heads, vd]; out [rows, heads, vd] of dtype; gate: logits of dtype, one per row
// and head, rows gate_stride apart, or null.
SOMI_API int somi_two_map_difference(const float* maps, float factor, float eps, float gain,
                                     const void* gate, long long gate_stride, long long rows, int heads,
                                     int vd, void* out, int dtype, cudaStream_t stream) {
    const long long n = rows * heads;
    if (n <= 0) return 0;
    if (vd <= 0) return SOMI_ERR_UNSUPPORTED;
    const int warps = 8;
    const long long want = (n + warps - 1) / warps;
    const int blocks = static_cast<int>(want < 148LL * 16 ? want : 148LL * 16);
    const TwoMaps two{factor, eps, gain, gate, gate_stride};
    if (dtype == SOMI_F32)
        launch_pdl(two_map_difference_kernel<float>, dim3(blocks), dim3(32 * warps), 0, stream, maps, two,
                   heads, vd, n, static_cast<float*>(out));
    else
        launch_pdl(two_map_difference_kernel<__nv_bfloat16>, dim3(blocks), dim3(32 * warps), 0, stream,
                   maps, two, heads, vd, n, static_cast<__nv_bfloat16*>(out));
    return launch_status();
}
