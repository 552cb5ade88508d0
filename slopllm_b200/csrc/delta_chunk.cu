// Chunked form of the gated delta rule with one decay per key channel (ops/delta.py) for portions of prompts, on the tensor cores.
//
// A sequence's tokens are cut into chunks of 64.  With b_t the running sum of the log decays inside a chunk, unit keys k and
//
//   A[t, s] = beta_t sum_c k_t[c] k_s[c] e^{b_t[c] - b_s[c]}   (s < t),      T = (I + A)^-1 diag(beta)
//
// the updates u of the chunk's tokens solve a triangular system, and
//
//   W = T (k e^b),   U0 = T v,   U = U0 - W S_in
//   S_out = diag(e^{b_C}) S_in + (k e^{b_C - b})^T U
//   o_t = (q_t e^{b_t}) . S_in + sum_{s<=t} [sum_c q_t[c] k_s[c] e^{b_t[c] - b_s[c]}] u_s
//
// in three launches:
//   1 delta_prepare_kernel  (chunk, head): decays, unit factors, A and its inverse, W, U0, the scores of q against k, and q and k
//                           with their decays
//   2 delta_scan_kernel     (value columns, head, sequence): carries the fp32 state over the chunks; leaves S_in and U of each
//   3 delta_output_kernel   (chunk, head): the two products of o, head norm, output gate
//
// No exponent is ever positive: e^{b_t - b_s} is taken directly inside 8-token diagonal blocks and through an anchor between the
// blocks elsewhere (token 31 between the halves, tokens 15 and 47 between the quarters, 7, 23, 39 and 55 inside those).  The inverse is fp32: 16 x 16 diagonal blocks by
// substitution, the others from products of blocks.  Every fp32 operand of a tensor-core product is split into two bf16 terms.
#include "gated_chunk.cuh"

namespace {

struct DeltaChunkParams {
    GatedScanParams s;                       // q, k, v behind the convolutions; g, out with strides of their own
    const int* chunks; const int* seq_chunks; int c0, c1;      // as in GatedChunkParams
    const float* z;                          // [T, h * dk]: raw decay input
    const float *dt_bias, *A_log;            // [h * dk], [h]
    const float* beta; int ld_beta;          // raw, [T, h]
    float unit_eps;
    // per (chunk of the pass, head); two terms: the high ones of all rows, then the low ones
    bf16 *w, *kt, *qt;                       // [2][CT][dk]: W, keys decayed to the end of the chunk, queries from its start
    bf16* pm;                                // [2][CT][CT]: scores
    float* decay;                            // [dk]: e^{b_C}
    float* u0;                               // [CT][dv]
    bf16* u;                                 // [2][CT][dv]
    bf16* sin;                               // [2][dk][dv]: S_in
    int stages;                              // set by the launcher: chunks of W and keys in shared memory
};

// max(x, 0) + log(1 + e^-|x|); the series keeps the relative accuracy of small values
__device__ __forceinline__ float softplus_f(float x) {
    const float t = __expf(-fabsf(x));
    const float series = t * (1.f - t * (0.5f - t * (0.33333333f - t * 0.25f)));
    return fmaxf(x, 0.f) + (t < 0.04f ? series : __logf(1.f + t));
}

constexpr int LDI = CT + 4, LDP = CT + 8;    // fp32 rows of A and of the inverse, bf16 rows of T and the scores

__device__ __forceinline__ int at_least(int a, int b) { return a > b ? a : b; }

size_t prepare_smem(int dk, int dv) {
    const int dkp = (dk + 15) / 16 * 16;
    const size_t a = (size_t)CT * LDI * 4, t2 = (size_t)2 * CT * LDP * 2, v = (size_t)CT * (dv + 8) * 2;
    return (size_t)2 * CT * (dkp + 8) * 2 + (size_t)CT * (dkp + 4) * 4 + (a > t2 ? a : t2) + (a > v ? a : v) + (size_t)3 * CT * 4;
}

// grid (chunks of the pass, h), block 256.  NP: pairs of key values per thread (dk <= 8 * NP).
template <int NP>
__global__ void __launch_bounds__(256, NP <= 16 ? 2 : 1) delta_prepare_kernel(DeltaChunkParams dp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    __shared__ int next_work;
    const GatedScanParams& p = dp.s;
    const int ci = blockIdx.x, h = blockIdx.y, hq = h / p.group, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int* ch = dp.chunks + (size_t)(dp.c0 + ci) * 4;
    const int t0 = ch[1], n = ch[2], dk = p.dk, dv = p.dv, dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8, ldb = dkp + 4;
    bf16* ks = reinterpret_cast<bf16*>(smraw);           // [CT][ldk] keys, then k e^b (high terms)
    bf16* qs = ks + CT * ldk;                            // [CT][ldk]
    float* bs = reinterpret_cast<float*>(qs + CT * ldk); // [CT][ldb] running log2 decays, then k e^b (low terms)
    float* A = bs + CT * ldb;                            // [CT][LDI], then T in two terms [2][CT][LDP]
    float* inv = A + at_least(CT * LDI, CT * LDP);       // [CT][LDI], then the values [CT][ldv]
    float *rk = inv + at_least(CT * LDI, CT * ldv / 2), *rq = rk + CT, *beta = rq + CT;
    const size_t base = (size_t)ci * p.h + h;
    load_rows(ks, ldk, (const bf16*)p.k + (size_t)t0 * p.ld + hq * dk, p.ld, n, dk, dkp);
    load_rows(qs, ldk, (const bf16*)p.q + (size_t)t0 * p.ld + hq * dk, p.ld, n, dk, dkp);
    cp_async_commit();
    const float rate = -expf(dp.A_log[h]) * LOG2E;
    const float* zb = dp.z + (size_t)t0 * (p.h * dk) + h * dk;
    for (int i = tid; i < CT * (dkp / 4); i += 256) {
        const int s = i / (dkp / 4), c = i % (dkp / 4) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s < n && c < dk) {
            const float4 z = *reinterpret_cast<const float4*>(zb + (size_t)s * (p.h * dk) + c);
            const float4 d = *reinterpret_cast<const float4*>(dp.dt_bias + h * dk + c);
            x = make_float4(rate * softplus_f(z.x + d.x), rate * softplus_f(z.y + d.y), rate * softplus_f(z.z + d.z), rate * softplus_f(z.w + d.w));
        }
        *reinterpret_cast<float4*>(bs + s * ldb + c) = x;
    }
    if (tid < CT) beta[tid] = tid < n ? sigmoid_f(dp.beta[(size_t)(t0 + tid) * dp.ld_beta + h]) : 0.f;
    if (tid == 0) next_work = 0;
    __syncthreads();
    // running sums: 16 tokens of a channel at a time, then what came before each
    for (int i = tid; i < 4 * dkp; i += 256) {
        const int c = i % dkp, s0 = i / dkp * 16;
        float run = 0.f;
#pragma unroll
        for (int s = 0; s < 16; ++s) {
            run += bs[(s0 + s) * ldb + c];
            bs[(s0 + s) * ldb + c] = run;
        }
    }
    cp_async_wait_all();
    __syncthreads();
    float before[4];                                     // (dkp <= 256: at most four pieces per thread)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = tid + j * 256;
        before[j] = 0.f;
        if (i < 4 * dkp)
            for (int q = 0; q < i / dkp; ++q) before[j] += bs[(q * 16 + 15) * ldb + i % dkp];
    }
    // unit factors: four lanes per token
    {
        const int s = tid >> 2;
        float a = 0.f, b = 0.f;
        for (int c = c4 * 2; c < dkp; c += 8) {          // (rows behind the chunk's end and padded columns are zero)
            const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + s * ldk + c)), y = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
            a += x.x * x.x + x.y * x.y;
            b += y.x * y.x + y.y * y.y;
        }
        a += __shfl_xor_sync(0xffffffffu, a, 1); a += __shfl_xor_sync(0xffffffffu, a, 2);
        b += __shfl_xor_sync(0xffffffffu, b, 1); b += __shfl_xor_sync(0xffffffffu, b, 2);
        if (c4 == 0) {
            rq[s] = s < n ? rsqrtf((float)dk) / sqrtf(a + dp.unit_eps) : 0.f;
            rk[s] = s < n ? 1.f / sqrtf(b + dp.unit_eps) : 0.f;
        }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int i = tid + j * 256;
        if (i < 4 * dkp && i >= dkp) {
            float* x = bs + (i / dkp * 16) * ldb + i % dkp;
#pragma unroll
            for (int s = 0; s < 16; ++s) x[s * ldb] += before[j];
        }
    }
    __syncthreads();
    bf16 *ph = dp.pm + base * 2 * CT * CT, *pl = ph + CT * CT;
    if (tid < dk) dp.decay[base * dk + tid] = exp2f(bs[(n - 1) * ldb + tid]);
    // ---- A and the scores outside the 16 x 16 diagonal blocks: a block per warp ----
    if (warp < 6) {
        const int bi = warp < 4 ? 2 + (warp >> 1) : warp == 4 ? 1 : 3, bj = warp < 4 ? (warp & 1) : warp == 4 ? 0 : 2;
        const int r0 = bi * 16 + g, r1 = r0 + 8;
        const float* an = bs + (warp < 4 ? 31 : bi * 16 - 1) * ldb;
        float aa[2][4] = {}, pp[2][4] = {};
        for (int kk = 0; kk < dkp; kk += 16) {
            uint32_t a[4], a2[4], q[4], q2[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = (i & 1) ? r1 : r0, c = kk + c4 * 2 + (i >> 1) * 8;
                const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c), o = *reinterpret_cast<const float2*>(an + c);
                const float ex = exp2_fast(fminf(b.x - o.x, 0.f)), ey = exp2_fast(fminf(b.y - o.y, 0.f));
                const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + r * ldk + c)), y = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                split_bf162(x.x * ex, x.y * ey, a[i], a2[i]);
                split_bf162(y.x * ex, y.y * ey, q[i], q2[i]);
            }
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                uint32_t bh[2], bl[2];
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int s = bj * 16 + t * 8 + g, c = kk + c4 * 2 + i * 8;
                    const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
                    const float2 b = *reinterpret_cast<const float2*>(bs + s * ldb + c), o = *reinterpret_cast<const float2*>(an + c);
                    split_bf162(x.x * exp2_fast(fminf(o.x - b.x, 0.f)), x.y * exp2_fast(fminf(o.y - b.y, 0.f)), bh[i], bl[i]);
                }
                mma_bf16_16816(aa[t], a, bh[0], bh[1]);
                mma_bf16_16816(pp[t], q, bh[0], bh[1]);
                mma_bf16_16816(aa[t], a, bl[0], bl[1]);
                mma_bf16_16816(pp[t], q, bl[0], bl[1]);
                mma_bf16_16816(aa[t], a2, bh[0], bh[1]);
                mma_bf16_16816(pp[t], q2, bh[0], bh[1]);
            }
        }
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = u ? r1 : r0, s = bj * 16 + t * 8 + c4 * 2;
                const float k0 = rk[s], k1 = rk[s + 1], fa = beta[r] * rk[r], fp = rq[r];
                *reinterpret_cast<float2*>(A + r * LDI + s) = make_float2(aa[t][u * 2] * fa * k0, aa[t][u * 2 + 1] * fa * k1);
                uint32_t hi, lo;
                split_bf162(pp[t][u * 2] * fp * k0, pp[t][u * 2 + 1] * fp * k1, hi, lo);
                *reinterpret_cast<uint32_t*>(ph + r * CT + s) = hi;
                *reinterpret_cast<uint32_t*>(pl + r * CT + s) = lo;
            }
    }
    // ---- the rest, to whoever is free: the lower left 8 x 8 quarters of the four diagonal blocks (rows 8 - 15 of a tile), then the
    //      pairs s <= r of eight 8 x 8 blocks, a quad of lanes per pair ----
    for (;;) {
        int it = 0;
        if (lane == 0) it = atomicAdd(&next_work, 1);
        it = __shfl_sync(0xffffffffu, it, 0);
        if (it >= 4 + 8 * 36 / 8) break;
        if (it < 4) {
            const int r = it * 16 + 8 + g;
            const float* an = bs + (it * 16 + 7) * ldb;
            float aa[4] = {}, pp[4] = {};
            for (int kk = 0; kk < dkp; kk += 16) {
                uint32_t a[4] = {}, a2[4] = {}, q[4] = {}, q2[4] = {}, bh[2], bl[2];
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int s = it * 16 + g, c = kk + c4 * 2 + i * 8;
                    const float2 o = *reinterpret_cast<const float2*>(an + c);
                    const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c), e = *reinterpret_cast<const float2*>(bs + s * ldb + c);
                    const float ex = exp2_fast(b.x - o.x), ey = exp2_fast(b.y - o.y);
                    const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + r * ldk + c)), y = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                    split_bf162(x.x * ex, x.y * ey, a[i * 2 + 1], a2[i * 2 + 1]);
                    split_bf162(y.x * ex, y.y * ey, q[i * 2 + 1], q2[i * 2 + 1]);
                    const float2 z = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
                    split_bf162(z.x * exp2_fast(o.x - e.x), z.y * exp2_fast(o.y - e.y), bh[i], bl[i]);
                }
                mma_bf16_16816(aa, a, bh[0], bh[1]);
                mma_bf16_16816(pp, q, bh[0], bh[1]);
                mma_bf16_16816(aa, a, bl[0], bl[1]);
                mma_bf16_16816(pp, q, bl[0], bl[1]);
                mma_bf16_16816(aa, a2, bh[0], bh[1]);
                mma_bf16_16816(pp, q2, bh[0], bh[1]);
            }
            const int s = it * 16 + c4 * 2;
            const float k0 = rk[s], k1 = rk[s + 1], fa = beta[r] * rk[r], fp = rq[r];
            *reinterpret_cast<float2*>(A + r * LDI + s) = make_float2(aa[2] * fa * k0, aa[3] * fa * k1);
            uint32_t hi, lo;
            split_bf162(pp[2] * fp * k0, pp[3] * fp * k1, hi, lo);
            *reinterpret_cast<uint32_t*>(ph + r * CT + s) = hi;
            *reinterpret_cast<uint32_t*>(pl + r * CT + s) = lo;
            *reinterpret_cast<uint32_t*>(ph + (r - 8) * CT + s + 8) = 0;             // (above the diagonal)
            *reinterpret_cast<uint32_t*>(pl + (r - 8) * CT + s + 8) = 0;
            continue;
        }
        const int y = (it - 4) * 8 + g, blk = y / 36, x = y % 36, i = x / 9, j = x % 9;      // rows i and 7 - i together have 9 pairs
        const int r = blk * 8 + (j <= i ? i : 7 - i), s = blk * 8 + (j <= i ? j : j - i - 1);
        float a0 = 0.f, a1 = 0.f, p0 = 0.f, p1 = 0.f;
        if (r < n) {
            const bf16 *kr = ks + r * ldk, *qr = qs + r * ldk, *k2 = ks + s * ldk;
            const float *br = bs + r * ldb, *b2 = bs + s * ldb;
#pragma unroll 4
            for (int c = c4 * 2; c < dk; c += 8) {
                const float2 x2 = bf162_to_f2(*reinterpret_cast<const uint32_t*>(kr + c)), q2 = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qr + c));
                const float2 y2 = bf162_to_f2(*reinterpret_cast<const uint32_t*>(k2 + c));
                const float2 u = *reinterpret_cast<const float2*>(br + c), v = *reinterpret_cast<const float2*>(b2 + c);
                const float ex = y2.x * exp2_fast(u.x - v.x), ey = y2.y * exp2_fast(u.y - v.y);
                a0 += x2.x * ex;
                a1 += x2.y * ey;
                p0 += q2.x * ex;
                p1 += q2.y * ey;
            }
        }
        float a = a0 + a1, q = p0 + p1;
        a += __shfl_xor_sync(0xffffffffu, a, 1); a += __shfl_xor_sync(0xffffffffu, a, 2);
        q += __shfl_xor_sync(0xffffffffu, q, 1); q += __shfl_xor_sync(0xffffffffu, q, 2);
        if (c4 == 0) {
            if (s < r) A[r * LDI + s] = a * beta[r] * rk[r] * rk[s];
            q *= rq[r] * rk[s];
            const bf16 hi = __float2bfloat16(q);
            ph[r * CT + s] = hi;
            pl[r * CT + s] = __float2bfloat16(q - __bfloat162float(hi));
            if (s != r) ph[s * CT + r] = pl[s * CT + r] = __float2bfloat16(0.f);
        }
    }
    __syncthreads();
    // ---- (I + A)^-1 ----
    if (warp < 4 && lane < 16) {
        const float* a = A + warp * 16 * LDI + warp * 16;
        float x[16];
#pragma unroll
        for (int r = 0; r < 16; ++r) {
            float v = r == lane ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < r; ++s) v -= a[r * LDI + s] * x[s];
            x[r] = v;
            inv[(warp * 16 + r) * LDI + warp * 16 + lane] = v;
        }
    }
    __syncthreads();
    for (int d = 1; d < 4; ++d) {                        // blocks (j + d, j); the block above the diagonal holds the inner sum
        const int r = tid >> 4, c = tid & 15;
        for (int j = 0; j + d < 4; ++j) {
            float m = 0.f;
            for (int k = j; k < j + d; ++k)
#pragma unroll
                for (int x = 0; x < 16; x += 4) {
                    const float4 y = *reinterpret_cast<const float4*>(A + ((j + d) * 16 + r) * LDI + k * 16 + x);
                    const float* z = inv + (k * 16 + x) * LDI + j * 16 + c;
                    m += y.x * z[0] + y.y * z[LDI] + y.z * z[2 * LDI] + y.w * z[3 * LDI];
                }
            inv[(j * 16 + r) * LDI + (j + d) * 16 + c] = m;
        }
        __syncthreads();
        for (int j = 0; j + d < 4; ++j) {
            const int i = j + d;
            float m = 0.f;
#pragma unroll
            for (int x = 0; x < 16; x += 4) {
                const float4 y = *reinterpret_cast<const float4*>(inv + (i * 16 + r) * LDI + i * 16 + x);
                const float* z = inv + (j * 16 + x) * LDI + i * 16 + c;
                m -= y.x * z[0] + y.y * z[LDI] + y.z * z[2 * LDI] + y.w * z[3 * LDI];
            }
            inv[(i * 16 + r) * LDI + j * 16 + c] = m;
        }
        __syncthreads();
    }
    bf16 *th = reinterpret_cast<bf16*>(A), *tl = th + CT * LDP;
    for (int i = tid; i < CT * CT / 2; i += 256) {
        const int t = i / (CT / 2), s = i % (CT / 2) * 2;
        uint32_t hi, lo;
        split_bf162(s <= t ? inv[t * LDI + s] * beta[s] : 0.f, s + 1 <= t ? inv[t * LDI + s + 1] * beta[s + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(th + t * LDP + s) = hi;
        *reinterpret_cast<uint32_t*>(tl + t * LDP + s) = lo;
    }
    __syncthreads();
    bf16* vs = reinterpret_cast<bf16*>(inv);
    load_rows(vs, ldv, (const bf16*)p.v + (size_t)t0 * p.ld + h * dv, p.ld, n, dv, dv);
    cp_async_commit();
    // ---- q and k with their decays: stored, and k e^b kept as the operand of W ----
    uint32_t wh[NP], wl[NP];
    const int per = dkp / 2;
    bf16 *kth = dp.kt + base * 2 * CT * dk, *qth = dp.qt + base * 2 * CT * dk;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
        const int i = tid + j * 256, s = i / per, c = i % per * 2;
        wh[j] = wl[j] = 0;
        if (s >= CT) continue;
        const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c)), y = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + s * ldk + c));
        const float2 b = *reinterpret_cast<const float2*>(bs + s * ldb + c), e = *reinterpret_cast<const float2*>(bs + (n - 1) * ldb + c);
        const float f = rk[s], fq = rq[s], ex = exp2_fast(b.x), ey = exp2_fast(b.y);
        split_bf162(x.x * f * ex, x.y * f * ey, wh[j], wl[j]);
        if (c < dk) {
            uint32_t hi, lo;
            split_bf162(x.x * f * exp2_fast(fminf(e.x - b.x, 0.f)), x.y * f * exp2_fast(fminf(e.y - b.y, 0.f)), hi, lo);
            *reinterpret_cast<uint32_t*>(kth + s * dk + c) = hi;
            *reinterpret_cast<uint32_t*>(kth + (CT + s) * dk + c) = lo;
            split_bf162(y.x * fq * ex, y.y * fq * ey, hi, lo);
            *reinterpret_cast<uint32_t*>(qth + s * dk + c) = hi;
            *reinterpret_cast<uint32_t*>(qth + (CT + s) * dk + c) = lo;
        }
    }
    __syncthreads();
    bf16* kl = reinterpret_cast<bf16*>(bs);              // [CT][ldk]
#pragma unroll
    for (int j = 0; j < NP; ++j) {
        const int i = tid + j * 256, s = i / per, c = i % per * 2;
        if (s >= CT) continue;
        *reinterpret_cast<uint32_t*>(ks + s * ldk + c) = wh[j];
        *reinterpret_cast<uint32_t*>(kl + s * ldk + c) = wl[j];
    }
    cp_async_wait_all();
    __syncthreads();
    // ---- W and U0: 16 tokens x 32 columns at a time ----
    const int rt = warp & 3, half = warp >> 2, r0 = rt * 16 + g, r1 = r0 + 8;
    bf16* wg = dp.w + base * 2 * CT * dk;
    float* ug = dp.u0 + base * CT * dv;
    for (int which = 0; which < 2; ++which) {
        const int cols = which == 0 ? dk : dv, ldx = which == 0 ? ldk : ldv;
        const bf16 *xh = which == 0 ? ks : vs, *xl = kl;
        for (int j0 = half * 32; j0 < cols; j0 += 64) {
            const int nt = min(4, (cols - j0) / 8);
            float acc[4][4] = {};
            for (int kk = 0; kk <= rt * 16; kk += 16) {
                uint32_t a[4], a2[4];
                ldsm_x4(a, th + (rt * 16 + (lane & 15)) * LDP + kk + (lane >> 4) * 8);
                ldsm_x4(a2, tl + (rt * 16 + (lane & 15)) * LDP + kk + (lane >> 4) * 8);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (i >= nt) break;
                    uint32_t b0, b1;
                    ldsm_x2_trans(b0, b1, xh + (kk + (lane & 15)) * ldx + j0 + i * 8);
                    mma_bf16_16816(acc[i], a, b0, b1);
                    mma_bf16_16816(acc[i], a2, b0, b1);
                    if (which == 0) {
                        ldsm_x2_trans(b0, b1, xl + (kk + (lane & 15)) * ldx + j0 + i * 8);
                        mma_bf16_16816(acc[i], a, b0, b1);
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                if (i >= nt) break;
                const int j = j0 + i * 8 + c4 * 2;
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int r = u ? r1 : r0;
                    if (which == 0) {
                        uint32_t hi, lo;
                        split_bf162(acc[i][u * 2], acc[i][u * 2 + 1], hi, lo);
                        *reinterpret_cast<uint32_t*>(wg + r * dk + j) = hi;
                        *reinterpret_cast<uint32_t*>(wg + (CT + r) * dk + j) = lo;
                    } else {
                        *reinterpret_cast<float2*>(ug + r * dv + j) = make_float2(acc[i][u * 2], acc[i][u * 2 + 1]);
                    }
                }
            }
        }
    }
}

// ---- 2: the state over the chunks --------------------------------------------------------------------------------------------
size_t scan_smem(int dk, int nt, int stages) {
    const int dkp = (dk + 15) / 16 * 16, lds = nt * 8 + 8;
    return ((size_t)stages * 4 * CT * (dkp + 8) + (size_t)2 * dkp * lds + (size_t)2 * CT * lds) * 2;
}

// B fragments (k = 16 rows from `row`, n = 8 * N columns from `col`) of a row-major bf16 tile
template <int N>
__device__ __forceinline__ void ldsm_b(uint32_t (&b)[N][2], const bf16* t, int ld, int row, int col) {
    const int lane = threadIdx.x & 31;
    if (N == 1) {
        ldsm_x2_trans(b[0][0], b[0][1], t + (row + (lane & 15)) * ld + col);
    } else {
#pragma unroll
        for (int x = 0; x + 1 < N; x += 2) {
            uint32_t v[4];
            ldsm_x4_trans(v, t + (row + (lane & 15)) * ld + col + x * 8 + (lane >> 4) * 8);
            b[x][0] = v[0]; b[x][1] = v[1]; b[x + 1][0] = v[2]; b[x + 1][1] = v[3];
        }
    }
}

// grid (ceil(dv / (8 * NT)), h, B), block 256.  MT: 16-row tiles of the state per warp (dk <= 128 * MT).  NT: 8-wide column tiles.
template <int MT, int NT>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaChunkParams dp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    constexpr int NH = NT / 2, LDS = NT * 8 + 8;
    const GatedScanParams& p = dp.s;
    const int j0 = blockIdx.x * NT * 8, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int lo = max(dp.seq_chunks[seq], dp.c0), hi = min(dp.seq_chunks[seq + 1], dp.c1), dk = p.dk, dv = p.dv;
    if (lo >= hi) return;
    const int dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, nn = min(NT, (dv - j0) / 8), tile = CT * ldk;
    bf16* wk = reinterpret_cast<bf16*>(smraw);           // stages x [W high | W low | keys high | keys low][CT][ldk]
    bf16* sh = wk + dp.stages * 4 * tile;                // [dkp][LDS] the state: high terms, low terms
    bf16* sl = sh + dkp * LDS;
    bf16* uh = sl + dkp * LDS;                           // [CT][LDS]
    bf16* ul = uh + CT * LDS;
    float* state = p.S + ((size_t)p.state_idx[seq] * p.h + h) * dk * dv + j0;
    float S[MT][NT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                const float2 x = r < dk && i < nn ? *reinterpret_cast<const float2*>(state + (size_t)r * dv + i * 8 + c4 * 2) : make_float2(0.f, 0.f);
                S[m][i][u * 2] = x.x;
                S[m][i][u * 2 + 1] = x.y;
            }
    const int pieces = dkp / 8;
    auto fetch = [&](int i) {
        if (i < hi) {
            const size_t base = ((size_t)(i - dp.c0) * p.h + h) * 2 * CT;
            bf16* dst = wk + (i - lo) % dp.stages * 4 * tile;
            for (int x = tid; x < 2 * CT * pieces; x += 256) {                       // rows of the high terms, then of the low ones
                const int r = x / pieces, c = x % pieces * 8;
                bf16* d = dst + r * ldk + c;
                if (c < dk) {
                    cp_async16(d, dp.w + (base + r) * dk + c);
                    cp_async16(d + 2 * tile, dp.kt + (base + r) * dk + c);
                } else {
                    *reinterpret_cast<uint4*>(d) = *reinterpret_cast<uint4*>(d + 2 * tile) = make_uint4(0, 0, 0, 0);
                }
            }
        }
        cp_async_commit();
    };
    const int rt = warp & 3, half = warp >> 2, r0 = rt * 16 + g, r1 = r0 + 8;
    float2 u0[NH][2];
    float keep[MT][2];
    auto ahead = [&](int i) {                            // what a chunk needs in registers
        const size_t at = (size_t)(i - dp.c0) * p.h + h;
#pragma unroll
        for (int x = 0; x < NH; ++x) {
            const bool in = half * NH + x < nn;
            const float* src = dp.u0 + at * CT * dv + j0 + (half * NH + x) * 8 + c4 * 2;
            u0[x][0] = in ? *reinterpret_cast<const float2*>(src + (size_t)r0 * dv) : make_float2(0.f, 0.f);
            u0[x][1] = in ? *reinterpret_cast<const float2*>(src + (size_t)r1 * dv) : make_float2(0.f, 0.f);
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                keep[m][u] = r < dk ? dp.decay[at * dk + r] : 0.f;
            }
    };
    fetch(lo);
    ahead(lo);
    for (int i = lo; i < hi; ++i) {
        const size_t at = (size_t)(i - dp.c0) * p.h + h;
        if (dp.stages > 1) fetch(i + 1);
        bf16 *gh = dp.sin + at * 2 * dk * dv + j0, *gl = gh + (size_t)dk * dv;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                if (r >= dkp) continue;
#pragma unroll
                for (int x = 0; x < NT; ++x) {
                    uint32_t wh, wl;
                    split_bf162(S[m][x][u * 2], S[m][x][u * 2 + 1], wh, wl);
                    *reinterpret_cast<uint32_t*>(sh + r * LDS + x * 8 + c4 * 2) = wh;
                    *reinterpret_cast<uint32_t*>(sl + r * LDS + x * 8 + c4 * 2) = wl;
                    if (r < dk && x < nn) {
                        *reinterpret_cast<uint32_t*>(gh + (size_t)r * dv + x * 8 + c4 * 2) = wh;
                        *reinterpret_cast<uint32_t*>(gl + (size_t)r * dv + x * 8 + c4 * 2) = wl;
                    }
                }
            }
        if (dp.stages > 1) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        const bf16* wt = wk + (i - lo) % dp.stages * 4 * tile;
        const bf16* kt = wt + 2 * tile;
        float acc[NH][3][4] = {};                        // the three products of a column tile do not wait for one another
#pragma unroll 2
        for (int kk = 0; kk < dkp; kk += 16) {
            uint32_t a[4], a2[4], b[NH][2], c[NH][2];
            ldsm_x4(a, wt + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
            ldsm_x4(a2, wt + tile + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
            ldsm_b<NH>(b, sh, LDS, kk, half * NH * 8);
            ldsm_b<NH>(c, sl, LDS, kk, half * NH * 8);
#pragma unroll
            for (int x = 0; x < NH; ++x) {
                mma_bf16_16816(acc[x][0], a, b[x][0], b[x][1]);
                mma_bf16_16816(acc[x][1], a, c[x][0], c[x][1]);
                mma_bf16_16816(acc[x][2], a2, b[x][0], b[x][1]);
            }
        }
        bf16* ug = dp.u + at * 2 * CT * dv + j0;
#pragma unroll
        for (int x = 0; x < NH; ++x)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = u ? r1 : r0, j = (half * NH + x) * 8 + c4 * 2;
                uint32_t wh, wl;
                split_bf162(u0[x][u].x - (acc[x][0][u * 2] + (acc[x][1][u * 2] + acc[x][2][u * 2])),
                            u0[x][u].y - (acc[x][0][u * 2 + 1] + (acc[x][1][u * 2 + 1] + acc[x][2][u * 2 + 1])), wh, wl);
                *reinterpret_cast<uint32_t*>(uh + r * LDS + j) = wh;
                *reinterpret_cast<uint32_t*>(ul + r * LDS + j) = wl;
                if (half * NH + x < nn) {
                    *reinterpret_cast<uint32_t*>(ug + (size_t)r * dv + j) = wh;
                    *reinterpret_cast<uint32_t*>(ug + (size_t)(CT + r) * dv + j) = wl;
                }
            }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int x = 0; x < NT; ++x) { S[m][x][0] *= keep[m][0]; S[m][x][1] *= keep[m][0]; S[m][x][2] *= keep[m][1]; S[m][x][3] *= keep[m][1]; }
        if (i + 1 < hi) ahead(i + 1);
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int row = (warp + m * 8) * 16;
            if (row >= dkp) continue;
#pragma unroll
            for (int ks = 0; ks < CT; ks += 16) {
                const int off = (ks + (lane & 7) + ((lane >> 4) & 1) * 8) * ldk + row + ((lane >> 3) & 1) * 8;
                uint32_t a[4], a2[4], b[NT][2], c[NT][2];
                ldsm_x4_trans(a, kt + off);
                ldsm_x4_trans(a2, kt + tile + off);
                ldsm_b<NT>(b, uh, LDS, ks, 0);
                ldsm_b<NT>(c, ul, LDS, ks, 0);
#pragma unroll
                for (int x = 0; x < NT; ++x) mma_bf16_16816(S[m][x], a, b[x][0], b[x][1]);
#pragma unroll
                for (int x = 0; x < NT; ++x) mma_bf16_16816(S[m][x], a, c[x][0], c[x][1]);
#pragma unroll
                for (int x = 0; x < NT; ++x) mma_bf16_16816(S[m][x], a2, b[x][0], b[x][1]);
            }
        }
        __syncthreads();
        if (dp.stages == 1) fetch(i + 1);
    }
    cp_async_wait_all();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < NT; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                if (r < dk && i < nn) *reinterpret_cast<float2*>(state + (size_t)r * dv + i * 8 + c4 * 2) = make_float2(S[m][i][u * 2], S[m][i][u * 2 + 1]);
            }
}

// ---- 3: outputs --------------------------------------------------------------------------------------------------------------
constexpr int SLAB = 64;                     // state rows in shared memory at a time (two slabs)

size_t delta_output_smem(int dk, int dv) {
    const int dkp = (dk + 15) / 16 * 16, ldv = dv + 8, rows = dkp < 2 * SLAB ? dkp : 2 * SLAB;
    const size_t slabs = (size_t)2 * rows * ldv, second = (size_t)2 * CT * LDP + (size_t)2 * CT * ldv;
    return ((size_t)2 * CT * (dkp + 8) + (slabs > second ? slabs : second)) * 2 + (size_t)CT * 4 * 4;
}

// grid (chunks of the pass, h), block 512: 4 row tiles of 16 tokens x 4 column quarters.  NT: 8-wide tiles per quarter.
template <int NT>
__global__ void __launch_bounds__(512, NT <= 4 ? 2 : 1) delta_output_kernel(DeltaChunkParams dp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const GatedScanParams& p = dp.s;
    const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int rt = warp & 3, quarter = warp >> 2;
    const int* ch = dp.chunks + (size_t)(dp.c0 + ci) * 4;
    const int t0 = ch[1], n = ch[2], dk = p.dk, dv = p.dv, dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8, rows = min(dkp, 2 * SLAB);
    const size_t base = (size_t)ci * p.h + h, slabs = (size_t)2 * rows * ldv, second = (size_t)2 * CT * LDP + (size_t)2 * CT * ldv;
    bf16* qh = reinterpret_cast<bf16*>(smraw);           // [2][CT][ldk]
    bf16* x = qh + 2 * CT * ldk;                         // [rows][2][ldv] the state; then scores [2][CT][LDP] and updates [2][CT][ldv]
    float* ssq = reinterpret_cast<float*>(x + (slabs > second ? slabs : second));
    // [rows][cols] of two terms from global memory, the low terms `lo` elements behind the high ones
    auto fetch = [&](bf16* dst, size_t dst_lo, int ld, const bf16* src, size_t src_lo, int nrows, int have, int cols, int padded) {
        const int per = padded / 8;
        for (int i = tid; i < nrows * per; i += 512) {
            const int r = i / per, c = i % per * 8;
            bf16* d = dst + r * ld + c;
            if (r < have && c < cols) {
                cp_async16(d, src + (size_t)r * cols + c);
                cp_async16(d + dst_lo, src + src_lo + (size_t)r * cols + c);
            } else {
                *reinterpret_cast<uint4*>(d) = *reinterpret_cast<uint4*>(d + dst_lo) = make_uint4(0, 0, 0, 0);
            }
        }
    };
    const bf16* sg = dp.sin + base * 2 * dk * dv;
    fetch(qh, CT * ldk, ldk, dp.qt + base * 2 * CT * dk, (size_t)CT * dk, CT, CT, dk, dkp);
    const int ntiles = dv / 8, tq = (ntiles + 3) / 4, nt0 = quarter * tq, ntn = max(0, min(tq, ntiles - nt0));
    const int r0 = rt * 16 + g, r1 = r0 + 8;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    auto product = [&](const bf16* ah, size_t a_lo, int lda, int a_col, const bf16* bh, size_t b_lo, int ldb, int steps) {
        for (int kk = 0; kk < steps; kk += 16) {
            uint32_t a[4], a2[4];
            ldsm_x4(a, ah + (rt * 16 + (lane & 15)) * lda + a_col + kk + (lane >> 4) * 8);
            ldsm_x4(a2, ah + a_lo + (rt * 16 + (lane & 15)) * lda + a_col + kk + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                if (i >= ntn) break;
                uint32_t b0, b1, l0, l1;
                ldsm_x2_trans(b0, b1, bh + (kk + (lane & 15)) * ldb + (nt0 + i) * 8);
                ldsm_x2_trans(l0, l1, bh + b_lo + (kk + (lane & 15)) * ldb + (nt0 + i) * 8);
                mma_bf16_16816(acc[i], a, b0, b1);
                mma_bf16_16816(acc[i], a, l0, l1);
                mma_bf16_16816(acc[i], a2, b0, b1);
            }
        }
    };
    for (int k0 = 0; k0 < dkp; k0 += rows) {
        const int m = min(rows, dkp - k0);
        if (k0 > 0) __syncthreads();
        fetch(x, (size_t)rows * ldv, ldv, sg + (size_t)k0 * dv, (size_t)dk * dv, m, dk - k0, dv, dv);
        cp_async_commit();
        cp_async_wait_all();
        __syncthreads();
        product(qh, CT * ldk, ldk, k0, x, (size_t)rows * ldv, ldv, m);
    }
    __syncthreads();
    bf16* us = x + 2 * CT * LDP;
    fetch(x, CT * LDP, LDP, dp.pm + base * 2 * CT * CT, (size_t)CT * CT, CT, CT, CT, CT);
    fetch(us, CT * ldv, ldv, dp.u + base * 2 * CT * dv, (size_t)CT * dv, CT, CT, dv, dv);
    cp_async_commit();
    cp_async_wait_all();
    __syncthreads();
    product(x, CT * LDP, LDP, 0, us, CT * ldv, ldv, rt * 16 + 16);
    float s0 = 0.f, s1 = 0.f;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        s0 += acc[i][0] * acc[i][0] + acc[i][1] * acc[i][1];
        s1 += acc[i][2] * acc[i][2] + acc[i][3] * acc[i][3];
    }
    s0 += __shfl_xor_sync(0xffffffffu, s0, 1); s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
    s1 += __shfl_xor_sync(0xffffffffu, s1, 1); s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
    if (c4 == 0) { ssq[r0 * 4 + quarter] = s0; ssq[r1 * 4 + quarter] = s1; }
    __syncthreads();
    const float i0 = rsqrtf((ssq[r0 * 4] + ssq[r0 * 4 + 1] + ssq[r0 * 4 + 2] + ssq[r0 * 4 + 3]) / (float)dv + p.eps);
    const float i1 = rsqrtf((ssq[r1 * 4] + ssq[r1 * 4 + 1] + ssq[r1 * 4 + 2] + ssq[r1 * 4 + 3]) / (float)dv + p.eps);
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        if (i >= ntn) break;
        const int j = (nt0 + i) * 8 + c4 * 2;
        const float2 w = make_float2(p.norm_w[j], p.norm_w[j + 1]);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = u ? r1 : r0;
            if (r >= n) continue;
            const float f = u ? i1 : i0;
            const float2 gt = bf162_to_f2(*reinterpret_cast<const uint32_t*>((const bf16*)p.g + (size_t)(t0 + r) * p.ldg + h * dv + j));
            *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)(t0 + r) * p.ldo + (size_t)h * dv + j) =
                f2_to_bf162(acc[i][u * 2] * f * w.x / (1.f + __expf(-gt.x)), acc[i][u * 2 + 1] * f * w.y / (1.f + __expf(-gt.y)));
        }
    }
}

}  // namespace

// 1 when the chunked kernels take these sizes (head rows of whole 16-byte pieces, tiles that fit in shared memory).
SL_API int sl_delta_chunk_ok(int dk, int dv) {
    if (dk < 8 || dv < 8 || dk % 8 != 0 || dv % 8 != 0 || dk > 256 || dv > 256) return 0;
    return prepare_smem(dk, dv) <= SMEM_MAX && scan_smem(dk, 4, 1) <= SMEM_MAX && delta_output_smem(dk, dv) <= SMEM_MAX;
}

// One pass over the chunks [c0, c1) of B sequences (bf16 rows in and out).  Passes of one step run in order on one stream.
SL_API int sl_delta_chunks(const DeltaChunkParams* args, int B, cudaStream_t s) {
    DeltaChunkParams params = *args;
    DeltaChunkParams* p = &params;
    const GatedScanParams& sp = p->s;
    if (B == 0 || p->c1 <= p->c0) return 0;
    if (!sl_delta_chunk_ok(sp.dk, sp.dv) || sp.ld % 8 != 0 || sp.ldg % 2 != 0 || sp.ldo % 2 != 0 || sp.group < 1 || B > 65535 || sp.h > 65535) return -1;
    if (((uintptr_t)sp.q | (uintptr_t)sp.k | (uintptr_t)sp.v | (uintptr_t)p->z | (uintptr_t)p->dt_bias) % 16 != 0 || ((uintptr_t)sp.g | (uintptr_t)sp.out) % 4 != 0)
        return -1;
    const int dk = sp.dk, dv = sp.dv, h = sp.h, nc = p->c1 - p->c0;
    const size_t s1 = prepare_smem(dk, dv), s3 = delta_output_smem(dk, dv);
    // narrow column slices while the wide ones would leave SMs idle (they read the chunk's operands more often)
    const int nt = dk <= 128 && (dv + 31) / 32 * h * B < 100 ? 2 : 4;
    p->stages = scan_smem(dk, nt, 2) <= SMEM_MAX ? 2 : 1;
    const size_t s2 = scan_smem(dk, nt, p->stages);
#define SL_RUN(KERN, GRID, THREADS, BYTES)                                                                         \
    {                                                                                                              \
        auto kern = KERN;                                                                                          \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(BYTES));                     \
        sl_launch(kern, GRID, THREADS, BYTES, s, *p);                                                              \
    }
    if (dk <= 128) SL_RUN(delta_prepare_kernel<16>, dim3(nc, h), 256, s1)
    else SL_RUN(delta_prepare_kernel<32>, dim3(nc, h), 256, s1)
    const dim3 grid((dv + nt * 8 - 1) / (nt * 8), h, B);
    if (nt == 2) SL_RUN((delta_scan_kernel<1, 2>), grid, 256, s2)
    else if (dk <= 128) SL_RUN((delta_scan_kernel<1, 4>), grid, 256, s2)
    else SL_RUN((delta_scan_kernel<2, 4>), grid, 256, s2)
    if (dv <= 128) SL_RUN(delta_output_kernel<4>, dim3(nc, h), 512, s3)
    else SL_RUN(delta_output_kernel<8>, dim3(nc, h), 512, s3)
#undef SL_RUN
    return SL_LAUNCH_CHECK();
}
