// Cosines and sines of a step's positions for every rotation of a model, made once per step and read by all its layers.
#include "common.cuh"

namespace {

// out[t, i] = (cos, sin) of positions[t] * freq[i].  The angle is reduced to a turn in fp64, so it keeps fp32 accuracy at any position.
// grid (ceil(n / 128), T), block 128
__global__ void __launch_bounds__(128) angle_table_kernel(float2* __restrict__ out, const int* __restrict__ positions, const double* __restrict__ freq, int n) {
    pdl_grid_sync();
    const int i = blockIdx.x * 128 + threadIdx.x, t = blockIdx.y;
    if (i >= n) return;
    constexpr double TURN = 6.283185307179586476925286766559;
    const double a = (double)positions[t] * freq[i];
    float s, c;
    sincosf((float)(a - TURN * rint(a / TURN)), &s, &c);
    out[(size_t)t * n + i] = make_float2(c, s);
}

}  // namespace

SL_API int sl_angle_table(void* out, const int* positions, const double* freq, int T, int n, cudaStream_t s) {
    if (T == 0 || n == 0) return 0;
    if (T > 65535) return -1;
    sl_launch(angle_table_kernel, dim3((n + 127) / 128, T), 128, 0, s, (float2*)out, positions, freq, n);
    return SL_LAUNCH_CHECK();
}
