// Gated delta rule with one decay per key channel, token by token (definition in ops/delta.py):
//
//   S = diag(g) S;  u = beta (v - S^T k);  S = S + k u^T;  o = S^T q;  out = rms(o) * w * sigmoid(g2 low_g)
//
// One block per (sequence, head).  The state stays in registers over the sequence's tokens (a thread holds four columns of every
// rg-th row), or in global memory for sizes that do not fit.  A decode step is one launch from the projections to the output
// projection's input: convolutions, unit norms, low-rank decay and gate, state update, head norm.  State, gates, norms and sums
// are fp32.
#include "common.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

struct DeltaStepParams {
    void* out; int ldo;                      // [T, ldo]: head h at h * dv
    const void *q, *k, *v; int ld;           // token-major rows; query / key head i at i * dk, value head i at i * dv
    const float* low; int ld_low, ra, rg;    // [T, ra (decay) | rg (gate)]
    const float* b;                          // [T, h] with the stride of `low`
    const void *a2, *g2;                     // [h * dk, ra], [h * dv, rg]
    const float *dt_bias, *A_log, *norm_w;   // [h * dk], [h], [dv]
    float eps, unit_eps;
    float* S;                                // [slots, h, dk, dv]
    const float* conv_w; float* conv; int taps;      // [taps, C], [slots, taps, C] (one token per sequence)
    const int* positions; const int* qo_indptr; const int* state_idx;
    int h, hk, dk, dv;
};

// NT threads.  ONE: one token per sequence, convolutions included (without it rows are convolved already).  MAXR > 0: dv % 4 == 0 and at most MAXR state rows per thread, in registers.  MAXR == 0: state in global memory.
template <int NT, int MAXR, bool ONE, typename TI, typename TO>
__global__ void __launch_bounds__(NT, ONE && NT == 512 && MAXR <= 8 ? 2 : 1) delta_step_kernel(DeltaStepParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    __shared__ float scratch[33], ss_q, ss_k;
    const int seq = blockIdx.x / p.h, h = blockIdx.x % p.h, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int t_begin = p.qo_indptr[seq], t_end = p.qo_indptr[seq + 1];
    if (t_begin >= t_end) return;
    const int dk = p.dk, dv = p.dv, group = p.h / p.hk, hk = h / group;
    constexpr int VW = MAXR > 0 ? 4 : 1, NR = MAXR > 0 ? MAXR : 1;
    const int nc = dv / VW, rg = nc >= NT ? 1 : NT / nc;          // column groups, row groups that share a column
    const int dkp = (dk + 3) / 4 * 4, dvp = (dv + 3) / 4 * 4;
    float *sq = sm, *sk = sq + dkp, *sa = sk + dkp, *sv = sa + dkp, *sg = sv + dvp, *slow = sg + dvp;
    float* part = slow + (p.ra + p.rg + 3) / 4 * 4;                 // [rg][dv]
    const int slot = p.state_idx[seq];
    float* S = p.S + ((size_t)slot * p.h + h) * dk * dv;
    const int c = tid % nc, r = tid / nc;
    const bool on = MAXR > 0 && r < rg;
    float4 st[NR];
    // the state is read when the first token's gates are done; until then it travels to L2 and takes no registers
    if (MAXR > 0)
        for (int i = tid * 32; i < dk * dv; i += NT * 32) prefetch_l2_line(S + i);
    // rows of a2 and g2 as 16-byte pieces
    const bool wide_low = sizeof(TO) == 2 && p.ra % 8 == 0 && p.rg % 8 == 0 && ((uintptr_t)p.a2 | (uintptr_t)p.g2) % 16 == 0;
    const float rate = expf(p.A_log[h]), qscale = 1.f / sqrtf((float)dk);
    for (int t = t_begin; ONE ? t == t_begin : t < t_end; ++t) {
        const TI* q = (const TI*)p.q + (size_t)t * p.ld + hk * dk;
        const TI* k = (const TI*)p.k + (size_t)t * p.ld + hk * dk;
        const TI* v = (const TI*)p.v + (size_t)t * p.ld + h * dv;
        const float* low = p.low + (size_t)t * p.ld_low;
        __syncthreads();
        for (int i = tid; i < p.ra + p.rg; i += NT) slow[i] = low[i];
        const int pos = p.positions[t];
        for (int i = tid; i < 2 * dk + dv; i += NT) {
            const TI* src = i < dk ? q + i : i < 2 * dk ? k + i - dk : v + i - 2 * dk;
            float x = to_f(*src);
            if (ONE) {
                const int C = 2 * p.hk * dk + p.h * dv;
                const int ch = i < dk ? hk * dk + i : i < 2 * dk ? (p.hk + hk) * dk + i - dk : 2 * p.hk * dk + h * dv + i - 2 * dk;
                float* ring = p.conv + (size_t)slot * p.taps * C + ch;
                float a = p.conv_w[(size_t)(p.taps - 1) * C + ch] * x;
#pragma unroll
                for (int j = 1; j < 4; ++j)
                    if (j < p.taps && j <= pos) a += p.conv_w[(size_t)(p.taps - 1 - j) * C + ch] * ring[(size_t)((pos - j) % p.taps) * C];
                for (int j = 4; j < p.taps && j <= pos; ++j)
                    a += p.conv_w[(size_t)(p.taps - 1 - j) * C + ch] * ring[(size_t)((pos - j) % p.taps) * C];
                // (nobody reads this row of the ring in this launch, so the heads that share the channel need no order)
                if (i >= 2 * dk || h % group == 0) ring[(size_t)(pos % p.taps) * C] = x;
                x = a * sigmoid_f(a);
            }
            (i < dk ? sq[i] : i < 2 * dk ? sk[i - dk] : sv[i - 2 * dk]) = x;
        }
        const float beta = sigmoid_f(p.b[(size_t)t * p.ld_low + h]);
        __syncthreads();
        if (warp < 2) {
            const float* x = warp == 0 ? sq : sk;
            float ss = 0.f;
            for (int i = lane; i < dk; i += 32) ss += x[i] * x[i];
            ss = warp_sum(ss);
            if (lane == 0) (warp == 0 ? ss_q : ss_k) = ss;
        }
        // low-rank decay and gate: four lanes per row
        for (int i0 = warp * 8; i0 < dk + dv; i0 += NT / 4) {
            const int i = i0 + (lane >> 2), c4 = lane & 3;
            const bool dec = i < dk, in = i < dk + dv;
            const int rank = !in ? 0 : dec ? p.ra : p.rg;
            const TO* w = dec ? (const TO*)p.a2 + (size_t)(h * dk + i) * rank : (const TO*)p.g2 + (size_t)(h * dv + i - dk) * rank;
            const float* x = dec ? slow : slow + p.ra;
            float z = 0.f;
            if (wide_low) {
#pragma unroll 4
                for (int j = c4 * 8; j < rank; j += 32) {
                    const uint4 v = *reinterpret_cast<const uint4*>(w + j);
                    const float2 a = bf162_to_f2(v.x), b = bf162_to_f2(v.y), c = bf162_to_f2(v.z), d = bf162_to_f2(v.w);
                    const float4 x0 = *reinterpret_cast<const float4*>(x + j), x1 = *reinterpret_cast<const float4*>(x + j + 4);
                    z += a.x * x0.x + a.y * x0.y + b.x * x0.z + b.y * x0.w + c.x * x1.x + c.y * x1.y + d.x * x1.z + d.y * x1.w;
                }
            } else {
                for (int j = c4; j < rank; j += 4) z += to_f(w[j]) * x[j];
            }
            z += __shfl_xor_sync(0xffffffffu, z, 1);
            z += __shfl_xor_sync(0xffffffffu, z, 2);
            if (c4 == 0 && in) {
                if (dec) sa[i] = expf(-rate * softplus_f(z + p.dt_bias[h * dk + i]));
                else sg[i - dk] = sigmoid_f(z);
            }
        }
        if (MAXR > 0 && t == t_begin) {
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int row = r + i * rg;
                st[i] = on && row < dk ? *reinterpret_cast<const float4*>(S + (size_t)row * dv + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
        __syncthreads();
        const float qs = qscale / sqrtf(ss_q + p.unit_eps), ks = 1.f / sqrtf(ss_k + p.unit_eps);
        if (MAXR > 0) {
            float4 kv = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int row = r + i * rg;
                if (row >= dk) break;
                const float a = sa[row], kk = sk[row];
                st[i].x *= a; st[i].y *= a; st[i].z *= a; st[i].w *= a;
                kv.x += st[i].x * kk; kv.y += st[i].y * kk; kv.z += st[i].z * kk; kv.w += st[i].w * kk;
            }
            if (on) *reinterpret_cast<float4*>(part + r * dv + c * 4) = kv;
            __syncthreads();
            float4 sum = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int i = 0; i < rg; ++i) {
                const float4 x = *reinterpret_cast<const float4*>(part + i * dv + c * 4);
                sum.x += x.x; sum.y += x.y; sum.z += x.z; sum.w += x.w;
            }
            const float4 vv = *reinterpret_cast<const float4*>(sv + c * 4);
            const float4 u = make_float4(beta * (vv.x - sum.x * ks) * ks, beta * (vv.y - sum.y * ks) * ks, beta * (vv.z - sum.z * ks) * ks,
                                         beta * (vv.w - sum.w * ks) * ks);
            __syncthreads();
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int i = 0; i < NR; ++i) {
                const int row = r + i * rg;
                if (row >= dk) break;
                const float kk = sk[row], qq = sq[row];
                st[i].x += kk * u.x; st[i].y += kk * u.y; st[i].z += kk * u.z; st[i].w += kk * u.w;
                o.x += st[i].x * qq; o.y += st[i].y * qq; o.z += st[i].z * qq; o.w += st[i].w * qq;
            }
            if (on) *reinterpret_cast<float4*>(part + r * dv + c * 4) = o;
        } else {
            for (int pass = 0; pass < 2; ++pass) {
                for (int c0 = 0; c0 < nc; c0 += NT) {
                    const int cc = nc >= NT ? c0 + tid : c, rr = nc >= NT ? 0 : r;
                    if (cc >= nc || rr >= rg) continue;
                    float acc = 0.f, u = 0.f;
                    if (pass == 1) u = sv[cc];                      // (the update, left there by the first pass)
                    for (int row = rr; row < dk; row += rg) {
                        float* x = S + (size_t)row * dv + cc;
                        const float s = pass == 0 ? *x * sa[row] : *x + sk[row] * u;
                        *x = s;
                        acc += s * (pass == 0 ? sk[row] : sq[row]);
                    }
                    part[rr * dv + cc] = acc;
                }
                __syncthreads();
                if (pass == 0) {
                    for (int j = tid; j < dv; j += NT) {
                        float sum = 0.f;
                        for (int i = 0; i < rg; ++i) sum += part[i * dv + j];
                        sv[j] = beta * (sv[j] - sum * ks) * ks;
                    }
                    __syncthreads();
                }
            }
        }
        __syncthreads();
        float ss = 0.f;
        for (int j = tid; j < dv; j += NT) {
            float o = 0.f;
            for (int i = 0; i < rg; ++i) o += part[i * dv + j];
            o *= qs;
            part[j] = o;                                            // (column j of every group was read by this thread alone)
            ss += o * o;
        }
        const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + p.eps);
        TO* out = (TO*)p.out + (size_t)t * p.ldo + (size_t)h * dv;
        for (int j = tid; j < dv; j += NT) put(out + j, part[j] * inv * p.norm_w[j] * sg[j]);
    }
    if (MAXR > 0 && on) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int row = r + i * rg;
            if (row < dk) *reinterpret_cast<float4*>(S + (size_t)row * dv + c * 4) = st[i];
        }
    }
}

}  // namespace

// in_f32: q, k, v rows are fp32 (else bf16); out_f32: `out`, a2 and g2 are fp32 (needs in_f32).  With `conv` every range has at
// most one token.
SL_API int sl_delta_step(const DeltaStepParams* p, int B, int in_f32, int out_f32, cudaStream_t s) {
    if (B == 0) return 0;
    if ((out_f32 && !in_f32) || p->dk < 1 || p->dv < 1 || p->hk < 1 || p->h % p->hk != 0 || (p->conv != nullptr && p->taps < 1)) return -1;
    const bool v4 = p->dv % 4 == 0 && p->dv <= 1024;
    auto rows = [&](int threads) { const int nc = p->dv / 4, rg = nc >= threads ? 1 : threads / nc; return (p->dk + rg - 1) / rg; };
    // as few state rows per thread as two blocks of 512 threads on an SM leave registers for
    const int threads = v4 && rows(256) > 8 ? 512 : 256, per = v4 ? rows(threads) : 0;
    const int maxr = !v4 ? 0 : per <= 4 ? 4 : per <= 8 ? 8 : per <= 16 ? 16 : 0;
    const int nc = maxr > 0 ? p->dv / 4 : p->dv, rg = nc >= threads ? 1 : threads / nc;
    const int low = (p->ra + p->rg + 3) / 4 * 4;
    const size_t smem = (size_t)(3 * ((p->dk + 3) / 4 * 4) + 2 * ((p->dv + 3) / 4 * 4) + low + rg * p->dv) * sizeof(float);
    if (smem > 200 * 1024) return -1;
#define SL_DS(N, R, TI, TO)                                                                                        \
    {                                                                                                              \
        auto kern = p->conv != nullptr ? delta_step_kernel<N, R, true, TI, TO> : delta_step_kernel<N, R, false, TI, TO>; \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
        sl_launch(kern, B * p->h, N, smem, s, *p);                                                                 \
    }
#define SL_DS_T(N, R)                                  \
    {                                                  \
        if (out_f32) SL_DS(N, R, float, float)         \
        else if (in_f32) SL_DS(N, R, float, bf16)      \
        else SL_DS(N, R, bf16, bf16)                   \
    }
    if (threads == 512) {
        if (maxr == 8 || maxr == 4) SL_DS_T(512, 8) else if (maxr == 16) SL_DS_T(512, 16) else SL_DS_T(512, 0)
    } else {
        if (maxr == 4) SL_DS_T(256, 4) else if (maxr == 8) SL_DS_T(256, 8) else SL_DS_T(256, 0)
    }
#undef SL_DS_T
#undef SL_DS
    return SL_LAUNCH_CHECK();
}
