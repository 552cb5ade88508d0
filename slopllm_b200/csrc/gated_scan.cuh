// Parameters and scalar functions shared by the step and chunk kernels of the gated outer-product recurrences.
#pragma once

#include "common.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float logsigmoid_f(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

enum { KIND_GLA = 0, KIND_MLSTM = 1, KIND_RETENTION = 2 };

struct GatedScanParams {
    void* out;                            // [T, h * dv]
    const void *q, *k, *v, *g; int ld;    // token-major rows with a common stride; head i at i * dk (q, k) or i * dv (v, g)
    const float* gates; int ld_gates;     // GLA: low-rank input [T, rank]; mLSTM: i_raw [T, h] | f_raw [T, h]
    const void* a2; const float* a2_b; int rank; float inv_tau;      // GLA: [h * dk, rank], [h * dk]
    const float *i_b, *f_b; float cap;    // mLSTM: [h]
    const float* norm_w;                  // GLA [dv], mLSTM [h * dv], retention: none
    float eps;
    float *S, *n, *m;                     // state
    const int* qo_indptr; const int* state_idx;
    int h, dk, dv;
    int ldg, ldo, group;                  // row stride of out; delta rule: row stride of g, heads that share a q / k head
    const float* decay;                   // retention: [2, h] decay of a head, its log2
    const float2* turn; int ldt, rot_dims;       // retention: (cos, sin) of pair m of token t at t * ldt + m; rotated values of a head
    float out_scale;                      // retention: factor on the output
};

// The adjacent values 2m, 2m + 1 of a query or key turned by the token's angle of pair m.
__device__ __forceinline__ float2 turned(const GatedScanParams& p, int t, int c, float2 x) {
    if (c >= p.rot_dims) return x;
    const float2 cs = p.turn[(size_t)t * p.ldt + (c >> 1)];
    return make_float2(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y);
}

}  // namespace
