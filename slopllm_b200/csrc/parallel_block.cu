// Activation of a feed-forward: act(gate + bias) * (up + bias), times the sigmoid of one number per row if the feed-forward is gated as
// a whole, or act(up) alone, from columns of a projection into columns of an operand.  Either may be part of wider rows: a feed-forward
// that runs beside a mixer shares its input and output product.
#include "common.cuh"

namespace {

enum { ACT_SILU = 0, ACT_GELU_TANH = 1 };

template <int ACT>
__device__ __forceinline__ float act_f(float g) {
    if (ACT == ACT_SILU) return g / (1.f + expf(-g));
    // 0.5 g (1 + tanh(x)) = g sigmoid(2x), x = sqrt(2 / pi) (g + 0.044715 g^3)
    return g / (1.f + expf(-1.5957691216057308f * (g + 0.044715f * g * g * g)));
}

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

// grid (ceil(I / (256 * VW)), T); bias [2 I] (gate | up) or null; row_gate [T] (elements ldg apart) or null
template <int ACT, int VW, typename TI, typename TO>
__global__ void __launch_bounds__(256) gated_act_rows_kernel(TO* __restrict__ out, int ldo, const TI* __restrict__ gu, int ld, const float* __restrict__ bias,
                                                             const float* __restrict__ row_gate, int ldg, int I) {
    pdl_grid_sync();
    const int i = (blockIdx.x * 256 + threadIdx.x) * VW, t = blockIdx.y;
    if (i >= I) return;
    const TI* g = gu + (size_t)t * ld + i;
    TO* o = out + (size_t)t * ldo + i;
    const float f = row_gate != nullptr ? 1.f / (1.f + expf(-row_gate[(size_t)t * ldg])) : 1.f;
    if (VW == 4) {
        float4 a = Four<TI>::load(g), b = Four<TI>::load(g + I);
        if (bias != nullptr) {
            const float4 x = Four<float>::load(bias + i), y = Four<float>::load(bias + I + i);
            a.x += x.x; a.y += x.y; a.z += x.z; a.w += x.w;
            b.x += y.x; b.y += y.y; b.z += y.z; b.w += y.w;
        }
        Four<TO>::store(o, make_float4(act_f<ACT>(a.x) * b.x * f, act_f<ACT>(a.y) * b.y * f, act_f<ACT>(a.z) * b.z * f, act_f<ACT>(a.w) * b.w * f));
    } else {
        float a = Four<TI>::one(g), b = Four<TI>::one(g + I);
        if (bias != nullptr) { a += bias[i]; b += bias[I + i]; }
        Four<TO>::put(o, act_f<ACT>(a) * b * f);
    }
}

// grid (ceil(I / (256 * VW)), T)
template <int ACT, int VW, typename TI, typename TO>
__global__ void __launch_bounds__(256) act_rows_kernel(TO* __restrict__ out, int ldo, const TI* __restrict__ x, int ld, int I) {
    pdl_grid_sync();
    const int i = (blockIdx.x * 256 + threadIdx.x) * VW, t = blockIdx.y;
    if (i >= I) return;
    const TI* g = x + (size_t)t * ld + i;
    TO* o = out + (size_t)t * ldo + i;
    if (VW == 4) {
        const float4 a = Four<TI>::load(g);
        Four<TO>::store(o, make_float4(act_f<ACT>(a.x), act_f<ACT>(a.y), act_f<ACT>(a.z), act_f<ACT>(a.w)));
    } else {
        Four<TO>::put(o, act_f<ACT>(Four<TI>::one(g)));
    }
}

struct ActArgs {
    void* out; int ldo;
    const void* x; int ld;               // [T, 2 I] (gate | up), or [T, I]
    const float *bias, *row_gate; int ldg;
    int T, I; bool gated;
};

template <int ACT, typename TI, typename TO>
int run(const ActArgs& a, cudaStream_t s) {
    const bool v4 = a.I % 4 == 0 && a.ldo % 4 == 0 && a.ld % 4 == 0 && (uintptr_t)a.out % (4 * sizeof(TO)) == 0 && (uintptr_t)a.x % (4 * sizeof(TI)) == 0;
    const dim3 grid((a.I / (v4 ? 4 : 1) + 255) / 256, a.T);
    TO* out = (TO*)a.out;
    const TI* x = (const TI*)a.x;
    if (a.gated && v4) sl_launch(gated_act_rows_kernel<ACT, 4, TI, TO>, grid, 256, 0, s, out, a.ldo, x, a.ld, a.bias, a.row_gate, a.ldg, a.I);
    else if (a.gated) sl_launch(gated_act_rows_kernel<ACT, 1, TI, TO>, grid, 256, 0, s, out, a.ldo, x, a.ld, a.bias, a.row_gate, a.ldg, a.I);
    else if (v4) sl_launch(act_rows_kernel<ACT, 4, TI, TO>, grid, 256, 0, s, out, a.ldo, x, a.ld, a.I);
    else sl_launch(act_rows_kernel<ACT, 1, TI, TO>, grid, 256, 0, s, out, a.ldo, x, a.ld, a.I);
    return SL_LAUNCH_CHECK();
}

template <int ACT>
int run_types(const ActArgs& a, int in_f32, int out_f32, cudaStream_t s) {
    if (out_f32) return run<ACT, float, float>(a, s);
    return in_f32 ? run<ACT, float, bf16>(a, s) : run<ACT, bf16, bf16>(a, s);
}

int run_act(const ActArgs& a, int act, int in_f32, int out_f32, cudaStream_t s) {
    if (a.T == 0 || a.I == 0) return 0;
    if (a.T > 65535 || (out_f32 && !in_f32)) return -1;
    if (act == ACT_SILU) return run_types<ACT_SILU>(a, in_f32, out_f32, s);
    return act == ACT_GELU_TANH ? run_types<ACT_GELU_TANH>(a, in_f32, out_f32, s) : -1;
}

}  // namespace

// act 0: silu, 1: the tanh form of gelu
SL_API int sl_gated_act_rows(void* out, int ldo, const void* gu, int ld, const float* bias, const float* row_gate, int ldg, int T, int I, int act, int in_f32,
                             int out_f32, cudaStream_t s) {
    return run_act({out, ldo, gu, ld, bias, row_gate, ldg, T, I, true}, act, in_f32, out_f32, s);
}

SL_API int sl_act_rows(void* out, int ldo, const void* x, int ld, int T, int I, int act, int in_f32, int out_f32, cudaStream_t s) {
    return run_act({out, ldo, x, ld, nullptr, nullptr, 0, T, I, false}, act, in_f32, out_f32, s);
}
