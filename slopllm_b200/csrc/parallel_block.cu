// Activation of a feed-forward that runs beside a mixer: silu(gate) * up from columns of a wider projection into columns of a
// wider operand, so that both sublayers share one input and one output product.
#include "common.cuh"

namespace {

__device__ __forceinline__ float silu_f(float g) { return g / (1.f + expf(-g)); }

template <typename T>
struct Four;
template <>
struct Four<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
    static __device__ __forceinline__ float one(const float* p) { return *p; }
    static __device__ __forceinline__ void put(float* p, float v) { *p = v; }
};
template <>
struct Four<bf16> {
    static __device__ __forceinline__ float4 load(const bf16* p) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const float2 a = bf162_to_f2(u.x), b = bf162_to_f2(u.y);
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(bf16* p, float4 v) {
        *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162(v.x, v.y), f2_to_bf162(v.z, v.w));
    }
    static __device__ __forceinline__ float one(const bf16* p) { return __bfloat162float(*p); }
    static __device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
};

// grid (ceil(I / (256 * VW)), T)
template <int VW, typename TI, typename TO>
__global__ void __launch_bounds__(256) silu_mul_rows_kernel(TO* __restrict__ out, int ldo, const TI* __restrict__ gu, int ld, int I) {
    pdl_grid_sync();
    const int i = (blockIdx.x * 256 + threadIdx.x) * VW, t = blockIdx.y;
    if (i >= I) return;
    const TI* g = gu + (size_t)t * ld + i;
    TO* o = out + (size_t)t * ldo + i;
    if (VW == 4) {
        const float4 a = Four<TI>::load(g), b = Four<TI>::load(g + I);
        Four<TO>::store(o, make_float4(silu_f(a.x) * b.x, silu_f(a.y) * b.y, silu_f(a.z) * b.z, silu_f(a.w) * b.w));
    } else {
        Four<TO>::put(o, silu_f(Four<TI>::one(g)) * Four<TI>::one(g + I));
    }
}

template <typename TI, typename TO>
int run(void* out, int ldo, const void* gu, int ld, int T, int I, cudaStream_t s) {
    const bool v4 = I % 4 == 0 && ldo % 4 == 0 && ld % 4 == 0 && (uintptr_t)out % (4 * sizeof(TO)) == 0 && (uintptr_t)gu % (4 * sizeof(TI)) == 0;
    if (v4) sl_launch(silu_mul_rows_kernel<4, TI, TO>, dim3((I / 4 + 255) / 256, T), 256, 0, s, (TO*)out, ldo, (const TI*)gu, ld, I);
    else sl_launch(silu_mul_rows_kernel<1, TI, TO>, dim3((I + 255) / 256, T), 256, 0, s, (TO*)out, ldo, (const TI*)gu, ld, I);
    return SL_LAUNCH_CHECK();
}

}  // namespace

SL_API int sl_silu_mul_rows(void* out, int ldo, const void* gu, int ld, int T, int I, int in_f32, int out_f32, cudaStream_t s) {
    if (T == 0 || I == 0) return 0;
    if (T > 65535 || (out_f32 && !in_f32)) return -1;
    if (out_f32) return run<float, float>(out, ldo, gu, ld, T, I, s);
    return in_f32 ? run<float, bf16>(out, ldo, gu, ld, T, I, s) : run<bf16, bf16>(out, ldo, gu, ld, T, I, s);
}
