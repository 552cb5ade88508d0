// Linear-attention recurrences with a gated outer-product state (sm_100a):
//
//   GLA    S_t = diag(alpha_t) S_{t-1} + k_t v_t^T,            o_t = S_t^T q_t
//          alpha = sigmoid(a2 . low + b)^(1/tau), one decay per key channel from a low-rank projection
//   mLSTM  m_t = max(f_t + m_{t-1}, i_t)
//          S_t = e^(f_t + m_{t-1} - m_t) S_{t-1} + e^(i_t - m_t) k_t v_t^T,  n_t likewise with k alone
//          o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6)
//          i = cap tanh((i_raw + b) / cap), f = logsigmoid(cap tanh((f_raw + b) / cap)), one each per head
//   retention  S_t = gamma S_{t-1} + k_t v_t^T,                o_t = S_t^T q_t
//          one fixed decay per head; queries and keys turn with their position (adjacent pairs, angles from a table)
//
// followed by the head's RMS norm, its weight (none for retention) and an output gate (silu, sigmoid for mLSTM).  State [slot, h, dk, dv]
// (and n [slot, h, dk], m [slot, h]), gates and accumulation are fp32; q is scaled by dk^-0.5.
//
//  * gated_step_kernel: one block per (sequence, head) walks the sequence's tokens with the state in global memory: the decode
//    step (one token: the state is read and written once, everything up to the output projection in one launch), and the path
//    for fp32 models and for sizes that the chunked kernels do not take.
#include "gated_scan.cuh"

namespace {

template <int KIND, int VW, typename TI, typename TO>
__global__ void __launch_bounds__(256) gated_step_kernel(GatedScanParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    __shared__ float scratch[33];
    const int seq = blockIdx.x / p.h, h = blockIdx.x % p.h, tid = threadIdx.x;
    const int t_begin = p.qo_indptr[seq], t_end = p.qo_indptr[seq + 1];
    if (t_begin >= t_end) return;
    const int dk = p.dk, dv = p.dv, nc = dv / VW;
    const int rg = nc >= 256 ? 1 : 256 / nc;             // row groups that share a column
    float* sq = sm;
    float* sk = sq + dk;
    float* sa = sk + dk;
    float* part = sa + dk;                               // [rg][dv]
    const size_t sh = (size_t)p.state_idx[seq] * p.h + h;
    float* S = p.S + sh * dk * dv;
    float* nv = KIND == KIND_MLSTM ? p.n + sh * dk : nullptr;
    float m = KIND == KIND_MLSTM ? p.m[sh] : 0.f;
    const float qscale = 1.f / sqrtf((float)dk);
    const float* nw = p.norm_w + (KIND == KIND_MLSTM ? (size_t)h * dv : 0);
    for (int t = t_begin; t < t_end; ++t) {
        const TI* q = (const TI*)p.q + (size_t)t * p.ld + h * dk;
        const TI* k = (const TI*)p.k + (size_t)t * p.ld + h * dk;
        const TI* v = (const TI*)p.v + (size_t)t * p.ld + h * dv;
        const TI* g = (const TI*)p.g + (size_t)t * p.ld + h * dv;
        float keep = KIND == KIND_RETENTION ? p.decay[h] : 1.f, add = 1.f;
        if (KIND == KIND_MLSTM) {
            const float* gr = p.gates + (size_t)t * p.ld_gates;
            const float gi = p.cap * tanhf((gr[h] + p.i_b[h]) / p.cap);
            const float gf = logsigmoid_f(p.cap * tanhf((gr[p.h + h] + p.f_b[h]) / p.cap));
            const float mn = fmaxf(gf + m, gi);
            keep = expf(gf + m - mn);
            add = expf(gi - mn);
            m = mn;
        }
        __syncthreads();
        for (int i = tid; i < dk; i += 256) {
            if (KIND == KIND_RETENTION) {
                float2 a = make_float2(to_f(q[i]), 0.f), b = make_float2(to_f(k[i]), 0.f);
                if (i < p.rot_dims) {
                    const int e = i & ~1;
                    a = turned(p, t, e, make_float2(to_f(q[e]), to_f(q[e + 1])));
                    b = turned(p, t, e, make_float2(to_f(k[e]), to_f(k[e + 1])));
                    if (i & 1) { a.x = a.y; b.x = b.y; }
                }
                sq[i] = a.x * qscale;
                sk[i] = b.x;
                continue;
            }
            sq[i] = to_f(q[i]) * qscale;
            sk[i] = to_f(k[i]);
            if (KIND == KIND_GLA) {
                const TO* a2 = (const TO*)p.a2 + (size_t)(h * dk + i) * p.rank;
                const float* lo = p.gates + (size_t)t * p.ld_gates;
                float z = p.a2_b[h * dk + i];
                for (int r = 0; r < p.rank; ++r) z += to_f(a2[r]) * lo[r];
                sa[i] = expf(logsigmoid_f(z) * p.inv_tau);
            }
        }
        __syncthreads();
        for (int c0 = 0; c0 < nc; c0 += 256) {
            const int c = c0 + (nc >= 256 ? tid : tid % nc), r = nc >= 256 ? 0 : tid / nc;
            if (c < nc && r < rg) {
                float vv[VW], acc[VW];
#pragma unroll
                for (int x = 0; x < VW; ++x) { vv[x] = to_f(v[c * VW + x]) * add; acc[x] = 0.f; }
#pragma unroll 8
                for (int i = r; i < dk; i += rg) {
                    float* ptr = S + (size_t)i * dv + c * VW;
                    const float a = KIND == KIND_GLA ? sa[i] : keep, kk = sk[i], qq = sq[i];
                    if (VW == 4) {
                        float4 s = *reinterpret_cast<const float4*>(ptr);
                        s.x = a * s.x + kk * vv[0]; s.y = a * s.y + kk * vv[1];
                        s.z = a * s.z + kk * vv[2]; s.w = a * s.w + kk * vv[3];
                        *reinterpret_cast<float4*>(ptr) = s;
                        acc[0] += s.x * qq; acc[1] += s.y * qq; acc[2] += s.z * qq; acc[3] += s.w * qq;
                    } else {
                        const float s = a * *ptr + kk * vv[0];
                        *ptr = s;
                        acc[0] += s * qq;
                    }
                }
#pragma unroll
                for (int x = 0; x < VW; ++x) part[r * dv + c * VW + x] = acc[x];
            }
        }
        float den = 1.f;
        if (KIND == KIND_MLSTM) {
            float nq = 0.f;
            for (int i = tid; i < dk; i += 256) {
                const float x = keep * nv[i] + add * sk[i];
                nv[i] = x;
                nq += x * sq[i];
            }
            den = 1.f / (fmaxf(fabsf(block_sum(nq, scratch)), expf(-m)) + 1e-6f);
        }
        __syncthreads();
        float ss = 0.f;
        for (int j = tid; j < dv; j += 256) {
            float o = 0.f;
            for (int r = 0; r < rg; ++r) o += part[r * dv + j];
            o *= den;
            part[j] = o;                                 // (column j of every group was read by this thread alone)
            ss += o * o;
        }
        const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)dv + p.eps);
        TO* out = (TO*)p.out + (size_t)t * p.ldo + h * dv;
        for (int j = tid; j < dv; j += 256) {
            const float gg = to_f(g[j]), act = KIND == KIND_MLSTM ? sigmoid_f(gg) : gg * sigmoid_f(gg);
            put(out + j, part[j] * inv * (KIND == KIND_RETENTION ? p.out_scale : nw[j]) * act);
        }
    }
    if (KIND == KIND_MLSTM && tid == 0) p.m[sh] = m;
}

template <int KIND, int VW>
int launch_step(const GatedScanParams* p, int B, int in_f32, int out_f32, size_t smem, cudaStream_t s) {
#define SL_STEP(TI, TO)                                                                                            \
    {                                                                                                              \
        auto kern = gated_step_kernel<KIND, VW, TI, TO>;                                                           \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
        sl_launch(kern, B * p->h, 256, smem, s, *p);                                                               \
    }
    if (out_f32) SL_STEP(float, float)
    else if (in_f32) SL_STEP(float, bf16)
    else SL_STEP(bf16, bf16)
#undef SL_STEP
    return SL_LAUNCH_CHECK();
}

}  // namespace

// kind 0: GLA, 1: mLSTM, 2: retention.  in_f32: q, k, v, g rows are fp32 (else bf16); out_f32: `out` and `a2` are fp32 (needs in_f32).
SL_API int sl_gated_step(const GatedScanParams* p, int B, int kind, int in_f32, int out_f32, cudaStream_t s) {
    if (B == 0) return 0;
    if ((out_f32 && !in_f32) || p->dk < 1 || p->dv < 1) return -1;
    const bool v4 = p->dv % 4 == 0;
    const int nc = v4 ? p->dv / 4 : p->dv, rg = nc >= 256 ? 1 : 256 / nc;
    const size_t smem = (size_t)(3 * p->dk + rg * p->dv) * sizeof(float);
    if (smem > 200 * 1024) return -1;
    if (kind == KIND_GLA) return v4 ? launch_step<KIND_GLA, 4>(p, B, in_f32, out_f32, smem, s) : launch_step<KIND_GLA, 1>(p, B, in_f32, out_f32, smem, s);
    if (kind == KIND_MLSTM) return v4 ? launch_step<KIND_MLSTM, 4>(p, B, in_f32, out_f32, smem, s) : launch_step<KIND_MLSTM, 1>(p, B, in_f32, out_f32, smem, s);
    if (kind == KIND_RETENTION && p->rot_dims <= p->dk && p->rot_dims % 2 == 0)
        return v4 ? launch_step<KIND_RETENTION, 4>(p, B, in_f32, out_f32, smem, s) : launch_step<KIND_RETENTION, 1>(p, B, in_f32, out_f32, smem, s);
    return -1;
}
