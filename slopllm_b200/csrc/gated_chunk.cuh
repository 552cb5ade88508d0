// What the chunked recurrences share (gated_chunk.cu: GLA and mLSTM, delta_chunk.cu: the gated delta rule).
#pragma once

#include "gated_scan.cuh"
#include "mma_sync.cuh"

namespace {

constexpr int CT = 64;                       // tokens per chunk

constexpr size_t SMEM_MAX = 220 * 1024, SMEM_TWO = 112 * 1024;       // one block per SM, two

// rows [n][dim] (bf16, 16-byte pieces) -> shared [CT][ld] with cp.async, zero beyond n rows and beyond dim columns up to `padded`
__device__ __forceinline__ void load_rows(bf16* dst, int ld, const bf16* src, size_t stride, int n, int dim, int padded) {
    const int per = padded / 8;
    for (int i = threadIdx.x; i < CT * per; i += blockDim.x) {
        const int r = i / per, c = (i % per) * 8;
        if (r < n && c < dim) cp_async16(dst + r * ld + c, src + (size_t)r * stride + c);
        else *reinterpret_cast<uint4*>(dst + r * ld + c) = make_uint4(0, 0, 0, 0);
    }
}

constexpr float LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

}  // namespace
