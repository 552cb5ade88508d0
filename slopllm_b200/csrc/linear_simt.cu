// Matrix products on the CUDA cores with fp32 accumulation: y[t, n] = sum_k x[t, k] W[n, k] for any shape and alignment.
// Serves models that run entirely in fp32 (no reduced-precision tensor-core mode touches their numbers) and bf16 shapes that
// the TMA-fed kernels do not take (rows that are not a multiple of 16 bytes).  Batched over heads through element strides.
#include "common.cuh"

namespace {

struct SimtLinearParams {
    void* y; const void* x; const void* w;
    int T, N, K, batch;
    long long y_t, y_b;              // element strides of y (column stride 1)
    long long x_t, x_b;              // ... of x
    long long w_n, w_k, w_b;         // ... of W
};

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

constexpr int TM = 64, TN = 64, TK = 16;

template <typename TI, typename TO>
__global__ void __launch_bounds__(256) linear_simt_kernel(SimtLinearParams p) {
    pdl_grid_sync();
    __shared__ float xs[TK][TM + 4], ws[TK][TN + 4];
    const int tid = threadIdx.x, n0 = blockIdx.x * TN, t0 = blockIdx.y * TM, b = blockIdx.z;
    const TI* x = (const TI*)p.x + b * p.x_b;
    const TI* w = (const TI*)p.w + b * p.w_b;
    TO* y = (TO*)p.y + b * p.y_b;
    const int tx = tid & 15, ty = tid >> 4;
    const bool k_fast = p.w_k == 1;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += TK) {
        for (int i = tid; i < TM * TK; i += 256) {
            const int r = i / TK, k = i % TK;
            xs[k][r] = (t0 + r < p.T && k0 + k < p.K) ? to_f(x[(t0 + r) * p.x_t + k0 + k]) : 0.f;
        }
        for (int i = tid; i < TN * TK; i += 256) {
            const int r = k_fast ? i / TK : i % TN, k = k_fast ? i % TK : i / TN;
            ws[k][r] = (n0 + r < p.N && k0 + k < p.K) ? to_f(w[(n0 + r) * p.w_n + (k0 + k) * p.w_k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < TK; ++k) {
            float a[4], c[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xs[k][ty * 4 + i]; c[i] = ws[k][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] += a[i] * c[j];
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int t = t0 + ty * 4 + i, n = n0 + tx * 4 + j;
            if (t < p.T && n < p.N) put(y + t * p.y_t + n, acc[i][j]);
        }
}

__global__ void silu_mul_f32_kernel(float* __restrict__ out, const float* __restrict__ gu, size_t total, int I) {
    pdl_grid_sync();
    for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
        const size_t t = idx / I, i = idx % I;
        const float g = gu[t * 2 * I + i], u = gu[t * 2 * I + I + i];
        out[idx] = g / (1.f + expf(-g)) * u;
    }
}

}  // namespace

// in_f32 / out_f32: element types of (x, W) and of y; in_f32 implies out_f32.
SL_API int sl_linear_simt(const SimtLinearParams* p, int in_f32, int out_f32, cudaStream_t s) {
    if (p->T <= 0 || p->N <= 0 || p->K <= 0 || p->batch <= 0) return 0;
    if ((in_f32 && !out_f32) || p->batch > 65535 || (p->T + TM - 1) / TM > 65535) return -1;
    const dim3 grid((p->N + TN - 1) / TN, (p->T + TM - 1) / TM, p->batch);
    if (in_f32) sl_launch(linear_simt_kernel<float, float>, grid, 256, 0, s, *p);
    else if (out_f32) sl_launch(linear_simt_kernel<bf16, float>, grid, 256, 0, s, *p);
    else sl_launch(linear_simt_kernel<bf16, bf16>, grid, 256, 0, s, *p);
    return SL_LAUNCH_CHECK();
}

// act[t, i] = silu(gu[t, i]) * gu[t, I + i] in fp32
SL_API int sl_silu_mul_f32(void* out, const void* gu, int T, int I, cudaStream_t s) {
    const size_t total = (size_t)T * I;
    if (total == 0) return 0;
    int blocks = (int)((total + 255) / 256);
    if (blocks > 148 * 16) blocks = 148 * 16;
    sl_launch(silu_mul_f32_kernel, blocks, 256, 0, s, (float*)out, (const float*)gu, total, I);
    return SL_LAUNCH_CHECK();
}
