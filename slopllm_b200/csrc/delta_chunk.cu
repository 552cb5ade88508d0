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
//   1 delta_prepare_kernel  (chunk, head): decays, unit factors, A and its inverse, W, U0, decayed keys
//   2 delta_scan_kernel     (value columns, head, sequence): carries the fp32 state over the chunks; leaves S_in and U of each
//   3 chunk_output_kernel   (chunk, head): gated_chunk.cuh, with U in the place of v
//
// No exponent is ever positive (see gated_chunk.cu).  The inverse is fp32: 16 x 16 diagonal blocks by substitution, the others
// from products of blocks.  Every other fp32 operand of a tensor-core product is split into two bf16 terms.
#include "gated_chunk.cuh"

namespace {

struct DeltaChunkParams {
    GatedChunkParams c;                      // c.b holds the decays' raw input z [T, h * dk] and then the running log2 decays
    const float *dt_bias, *A_log;            // [h * dk], [h]
    const float* beta; int ld_beta;          // raw, [T, h]
    float unit_eps;
    bf16* w;                                 // [chunks of the pass, h, high | low, CT, dk]
    bf16* kt;                                // decayed keys, likewise
    float* u0;                               // [chunks of the pass, h, CT, dv]
    bf16* u;                                 // [chunks of the pass, h, high | low, CT, dv]
    float* unit;                             // [T, h, 2]
    int stages;                              // set by the launcher: chunks of W and keys in shared memory
};

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

constexpr int LDI = CT + 4;                  // fp32 rows of A and of the inverse

size_t prepare_smem(int dk, int dv) {
    const int dkp = (dk + 15) / 16 * 16;
    const size_t a = (size_t)CT * LDI * 4, t2 = (size_t)2 * CT * LDA * 2;
    return (size_t)CT * (dkp + 8) * 2 + (size_t)CT * (dv + 8) * 2 + (size_t)CT * (dkp + 4) * 4 + (a > t2 ? a : t2) + a + (size_t)3 * CT * 4;
}

// grid (chunks of the pass, h), block 256.  NP: pairs of key values per thread (dk <= 8 * NP).
template <int NP>
__global__ void __launch_bounds__(256, NP <= 16 ? 2 : 1) delta_prepare_kernel(DeltaChunkParams dp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const GatedChunkParams& cp = dp.c;
    const GatedScanParams& p = cp.s;
    const int ci = blockIdx.x, h = blockIdx.y, hq = h / p.group, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int* ch = cp.chunks + (size_t)(cp.c0 + ci) * 4;
    const int t0 = ch[1], n = ch[2], dk = p.dk, dv = p.dv, dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8, ldb = dkp + 4;
    bf16* ks = reinterpret_cast<bf16*>(smraw);           // [CT][ldk] keys, then k e^b (high terms)
    bf16* vs = ks + CT * ldk;                            // [CT][ldv]
    float* bs = reinterpret_cast<float*>(vs + CT * ldv); // [CT][ldb] running log2 decays, then k e^b (low terms)
    float* A = bs + CT * ldb;                            // [CT][LDI], then T in two terms [2][CT][LDA]
    float* inv = A + (CT * LDI > CT * LDA ? CT * LDI : CT * LDA);      // [CT][LDI]
    float *rk = inv + CT * LDI, *rq = rk + CT, *beta = rq + CT;
    const int ldz = p.h * dk;
    float* zb = cp.b + (size_t)t0 * ldz + h * dk;
    load_rows(ks, ldk, (const bf16*)p.k + (size_t)t0 * p.ld + hq * dk, p.ld, n, dk, dkp);
    load_rows(vs, ldv, (const bf16*)p.v + (size_t)t0 * p.ld + h * dv, p.ld, n, dv, dv);
    cp_async_commit();
    const float rate = -expf(dp.A_log[h]) * LOG2E;
    for (int i = tid; i < CT * (dkp / 4); i += 256) {
        const int s = i / (dkp / 4), c = i % (dkp / 4) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s < n && c < dk) {
            const float4 z = *reinterpret_cast<const float4*>(zb + (size_t)s * ldz + c);
            const float4 d = *reinterpret_cast<const float4*>(dp.dt_bias + h * dk + c);
            x = make_float4(rate * softplus_f(z.x + d.x), rate * softplus_f(z.y + d.y), rate * softplus_f(z.z + d.z), rate * softplus_f(z.w + d.w));
        }
        *reinterpret_cast<float4*>(bs + s * ldb + c) = x;
    }
    if (tid < CT) beta[tid] = tid < n ? sigmoid_f(dp.beta[(size_t)(t0 + tid) * dp.ld_beta + h]) : 0.f;
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
    // unit factors, a warp per token (n <= CT)
    const float qscale = rsqrtf((float)dk);
    for (int s = warp; s < CT; s += 8) {
        float a = 0.f, b = 0.f;
        if (s < n) {
            const bf16* q = (const bf16*)p.q + (size_t)(t0 + s) * p.ld + hq * dk;
            for (int c = lane * 2; c < dk; c += 64) {
                const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(q + c)), y = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
                a += x.x * x.x + x.y * x.y;
                b += y.x * y.x + y.y * y.y;
            }
        }
        a = warp_sum(a);
        b = warp_sum(b);
        if (lane == 0) {
            rq[s] = s < n ? qscale / sqrtf(a + dp.unit_eps) : 0.f;
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
    if (tid < n) *reinterpret_cast<float2*>(dp.unit + ((size_t)(t0 + tid) * p.h + h) * 2) = make_float2(rq[tid], rk[tid]);
    __syncthreads();
    for (int i = tid; i < n * (dk / 4); i += 256) {
        const int s = i / (dk / 4), c = i % (dk / 4) * 4;
        *reinterpret_cast<float4*>(zb + (size_t)s * ldz + c) = *reinterpret_cast<const float4*>(bs + s * ldb + c);
    }
    // ---- A below the diagonal blocks: 16 x 8 pieces over the warps, decays through the row in front of the row block ----
    for (int u = warp; u < 12; u += 8) {
        const int pair = u >> 1, bi = pair == 0 ? 1 : pair <= 2 ? 2 : 3, bj = pair == 0 ? 0 : pair <= 2 ? pair - 1 : pair - 3;
        const int r0 = bi * 16 + g, r1 = r0 + 8, s = bj * 16 + (u & 1) * 8;
        const float* an = bs + (bi * 16 - 1) * ldb;
        float acc[4] = {};
        for (int kk = 0; kk < dkp; kk += 16) {
            uint32_t a[4], a2[4], bh[2], bl[2];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const int r = (i & 1) ? r1 : r0, c = kk + c4 * 2 + (i >> 1) * 8;
                const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + r * ldk + c));
                const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c), o = *reinterpret_cast<const float2*>(an + c);
                split_bf162(x.x * exp2_fast(fminf(b.x - o.x, 0.f)), x.y * exp2_fast(fminf(b.y - o.y, 0.f)), a[i], a2[i]);
            }
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                const int c = kk + c4 * 2 + i * 8;
                const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + (s + g) * ldk + c));
                const float2 b = *reinterpret_cast<const float2*>(bs + (s + g) * ldb + c), o = *reinterpret_cast<const float2*>(an + c);
                split_bf162(x.x * exp2_fast(fminf(o.x - b.x, 0.f)), x.y * exp2_fast(fminf(o.y - b.y, 0.f)), bh[i], bl[i]);
            }
            mma_bf16_16816(acc, a, bh[0], bh[1]);
            mma_bf16_16816(acc, a, bl[0], bl[1]);
            mma_bf16_16816(acc, a2, bh[0], bh[1]);
        }
        const int sc = s + c4 * 2;
        const float f0 = beta[r0] * rk[r0], f1 = beta[r1] * rk[r1];
        A[r0 * LDI + sc] = acc[0] * f0 * rk[sc];
        A[r0 * LDI + sc + 1] = acc[1] * f0 * rk[sc + 1];
        A[r1 * LDI + sc] = acc[2] * f1 * rk[sc];
        A[r1 * LDI + sc + 1] = acc[3] * f1 * rk[sc + 1];
    }
    // ---- diagonal blocks: the 120 pairs s < r of each, a quad of lanes per pair ----
    for (int it = tid >> 2; it < 4 * 120; it += 64) {
        const int blk = it / 120, x = it % 120, i = x / 15, j = x % 15;              // rows i and 15 - i together have 15 pairs
        const int r = blk * 16 + (j < i ? i : 15 - i), s = blk * 16 + (j < i ? j : j - i);
        float a0 = 0.f, a1 = 0.f;
        if (r < n) {
#pragma unroll 4
            for (int c = c4 * 2; c < dk; c += 8) {
                const float2 x2 = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + r * ldk + c));
                const float2 y2 = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
                const float2 br = *reinterpret_cast<const float2*>(bs + r * ldb + c), b2 = *reinterpret_cast<const float2*>(bs + s * ldb + c);
                a0 += x2.x * y2.x * exp2_fast(br.x - b2.x);
                a1 += x2.y * y2.y * exp2_fast(br.y - b2.y);
            }
        }
        float a = a0 + a1;
        a += __shfl_xor_sync(0xffffffffu, a, 1);
        a += __shfl_xor_sync(0xffffffffu, a, 2);
        if (c4 == 0) A[r * LDI + s] = a * beta[r] * rk[r] * rk[s];
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
                for (int x = 0; x < 16; ++x) m += A[((j + d) * 16 + r) * LDI + k * 16 + x] * inv[(k * 16 + x) * LDI + j * 16 + c];
            inv[(j * 16 + r) * LDI + (j + d) * 16 + c] = m;
        }
        __syncthreads();
        for (int j = 0; j + d < 4; ++j) {
            const int i = j + d;
            float m = 0.f;
#pragma unroll
            for (int x = 0; x < 16; ++x) m -= inv[(i * 16 + r) * LDI + i * 16 + x] * inv[(j * 16 + x) * LDI + i * 16 + c];
            inv[(i * 16 + r) * LDI + j * 16 + c] = m;
        }
        __syncthreads();
    }
    bf16 *th = reinterpret_cast<bf16*>(A), *tl = th + CT * LDA;
    for (int i = tid; i < CT * CT / 2; i += 256) {
        const int t = i / (CT / 2), s = i % (CT / 2) * 2;
        uint32_t hi, lo;
        split_bf162(s <= t ? inv[t * LDI + s] * beta[s] : 0.f, s + 1 <= t ? inv[t * LDI + s + 1] * beta[s + 1] : 0.f, hi, lo);
        *reinterpret_cast<uint32_t*>(th + t * LDA + s) = hi;
        *reinterpret_cast<uint32_t*>(tl + t * LDA + s) = lo;
    }
    // ---- decayed keys: to the end of the chunk (stored), from its start (operand of W) ----
    const size_t base = (size_t)ci * p.h + h;
    uint32_t wh[NP], wl[NP];
    const int per = dkp / 2;
#pragma unroll
    for (int j = 0; j < NP; ++j) {
        const int i = tid + j * 256, s = i / per, c = i % per * 2;
        wh[j] = wl[j] = 0;
        if (s >= CT) continue;
        const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
        const float2 b = *reinterpret_cast<const float2*>(bs + s * ldb + c), e = *reinterpret_cast<const float2*>(bs + (n - 1) * ldb + c);
        const float f = rk[s];
        split_bf162(x.x * f * exp2_fast(b.x), x.y * f * exp2_fast(b.y), wh[j], wl[j]);
        uint32_t hi, lo;
        split_bf162(x.x * f * exp2_fast(fminf(e.x - b.x, 0.f)), x.y * f * exp2_fast(fminf(e.y - b.y, 0.f)), hi, lo);
        if (c < dk) {
            *reinterpret_cast<uint32_t*>(dp.kt + (base * 2 * CT + s) * dk + c) = hi;
            *reinterpret_cast<uint32_t*>(dp.kt + ((base * 2 + 1) * CT + s) * dk + c) = lo;
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
    __syncthreads();
    // ---- W and U0: 16 tokens x 32 columns at a time ----
    const int rt = warp & 3, half = warp >> 2, r0 = rt * 16 + g, r1 = r0 + 8;
    for (int which = 0; which < 2; ++which) {
        const int cols = which == 0 ? dk : dv, ldx = which == 0 ? ldk : ldv;
        const bf16 *xh = which == 0 ? ks : vs, *xl = kl;
        for (int j0 = half * 32; j0 < cols; j0 += 64) {
            const int nt = min(4, (cols - j0) / 8);
            float acc[4][4] = {};
            for (int kk = 0; kk <= rt * 16; kk += 16) {
                uint32_t a[4], a2[4];
                ldsm_x4(a, th + (rt * 16 + (lane & 15)) * LDA + kk + (lane >> 4) * 8);
                ldsm_x4(a2, tl + (rt * 16 + (lane & 15)) * LDA + kk + (lane >> 4) * 8);
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
                if (which == 0) {
                    uint32_t hi, lo;
                    split_bf162(acc[i][0], acc[i][1], hi, lo);
                    *reinterpret_cast<uint32_t*>(dp.w + (base * 2 * CT + r0) * dk + j) = hi;
                    *reinterpret_cast<uint32_t*>(dp.w + ((base * 2 + 1) * CT + r0) * dk + j) = lo;
                    split_bf162(acc[i][2], acc[i][3], hi, lo);
                    *reinterpret_cast<uint32_t*>(dp.w + (base * 2 * CT + r1) * dk + j) = hi;
                    *reinterpret_cast<uint32_t*>(dp.w + ((base * 2 + 1) * CT + r1) * dk + j) = lo;
                } else {
                    *reinterpret_cast<float2*>(dp.u0 + (base * CT + r0) * dv + j) = make_float2(acc[i][0], acc[i][1]);
                    *reinterpret_cast<float2*>(dp.u0 + (base * CT + r1) * dv + j) = make_float2(acc[i][2], acc[i][3]);
                }
            }
        }
    }
}

// ---- 2: the state over the chunks --------------------------------------------------------------------------------------------
constexpr int NV = 32, LDS = NV + 8;         // value columns per block

size_t scan_smem(int dk, int stages) {
    const int dkp = (dk + 15) / 16 * 16;
    return ((size_t)stages * 4 * CT * (dkp + 8) + (size_t)2 * dkp * LDS + (size_t)2 * CT * LDS) * 2;
}

// grid (ceil(dv / NV), h, B), block 256.  MT: 16-row tiles of the state per warp (dk <= 128 * MT).
template <int MT>
__global__ void __launch_bounds__(256) delta_scan_kernel(DeltaChunkParams dp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const GatedChunkParams& cp = dp.c;
    const GatedScanParams& p = cp.s;
    const int j0 = blockIdx.x * NV, h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int lo = max(cp.seq_chunks[seq], cp.c0), hi = min(cp.seq_chunks[seq + 1], cp.c1), dk = p.dk, dv = p.dv;
    if (lo >= hi) return;
    const int dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, nn = min(NV / 8, (dv - j0) / 8), tile = CT * ldk;
    bf16* wk = reinterpret_cast<bf16*>(smraw);           // stages x [W high | W low | keys high | keys low][CT][ldk]
    bf16* sh = wk + dp.stages * 4 * tile;                // [dkp][LDS] the state: high terms, low terms
    bf16* sl = sh + dkp * LDS;
    bf16* uh = sl + dkp * LDS;                           // [CT][LDS]
    bf16* ul = uh + CT * LDS;
    float* state = p.S + ((size_t)p.state_idx[seq] * p.h + h) * dk * dv + j0;
    float S[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                const float2 x = r < dk && i < nn ? *reinterpret_cast<const float2*>(state + (size_t)r * dv + i * 8 + c4 * 2) : make_float2(0.f, 0.f);
                S[m][i][u * 2] = x.x;
                S[m][i][u * 2 + 1] = x.y;
            }
    auto fetch = [&](int i) {
        if (i < hi) {
            const size_t base = ((size_t)(i - cp.c0) * p.h + h) * 2 * CT;
            bf16* dst = wk + (i - lo) % dp.stages * 4 * tile;
            load_rows(dst, ldk, dp.w + base * dk, dk, CT, dk, dkp);
            load_rows(dst + tile, ldk, dp.w + (base + CT) * dk, dk, CT, dk, dkp);
            load_rows(dst + 2 * tile, ldk, dp.kt + base * dk, dk, CT, dk, dkp);
            load_rows(dst + 3 * tile, ldk, dp.kt + (base + CT) * dk, dk, CT, dk, dkp);
        }
        cp_async_commit();
    };
    const int rt = warp & 3, half = warp >> 2, r0 = rt * 16 + g, r1 = r0 + 8;
    fetch(lo);
    for (int i = lo; i < hi; ++i) {
        const size_t at = (size_t)(i - cp.c0) * p.h + h;
        const int* ch = cp.chunks + (size_t)i * 4;
        if (dp.stages > 1) fetch(i + 1);
        float2 u0[2][2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int j = (half * 2 + x) * 8;
            const bool in = half * 2 + x < nn;
            const float* src = dp.u0 + at * CT * dv + j0 + j + c4 * 2;
            u0[x][0] = in ? *reinterpret_cast<const float2*>(src + (size_t)r0 * dv) : make_float2(0.f, 0.f);
            u0[x][1] = in ? *reinterpret_cast<const float2*>(src + (size_t)r1 * dv) : make_float2(0.f, 0.f);
        }
        float keep[MT][2];
        const float* bc = cp.b + (size_t)(ch[1] + ch[2] - 1) * (p.h * dk) + h * dk;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                keep[m][u] = r < dk ? bc[r] : 0.f;
            }
        bf16* sin = reinterpret_cast<bf16*>(cp.loc + at * dk * dv);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                if (r >= dkp) continue;
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    uint32_t wh, wl;
                    split_bf162(S[m][x][u * 2], S[m][x][u * 2 + 1], wh, wl);
                    *reinterpret_cast<uint32_t*>(sh + r * LDS + x * 8 + c4 * 2) = wh;
                    *reinterpret_cast<uint32_t*>(sl + r * LDS + x * 8 + c4 * 2) = wl;
                    if (r < dk && x < nn) {              // eight high terms, then their eight low terms
                        bf16* dst = sin + ((size_t)r * dv + j0 + x * 8) * 2 + c4 * 2;
                        *reinterpret_cast<uint32_t*>(dst) = wh;
                        *reinterpret_cast<uint32_t*>(dst + 8) = wl;
                    }
                }
            }
        if (dp.stages > 1) cp_async_wait<1>();
        else cp_async_wait<0>();
        __syncthreads();
        const bf16* wt = wk + (i - lo) % dp.stages * 4 * tile;
        const bf16* kt = wt + 2 * tile;
        float acc[2][4] = {};
        for (int kk = 0; kk < dkp; kk += 16) {
            uint32_t a[4], a2[4], b[4], c[4];
            ldsm_x4(a, wt + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
            ldsm_x4(a2, wt + tile + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
            ldsm_x4_trans(b, sh + (kk + (lane & 15)) * LDS + half * 16 + (lane >> 4) * 8);
            ldsm_x4_trans(c, sl + (kk + (lane & 15)) * LDS + half * 16 + (lane >> 4) * 8);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                mma_bf16_16816(acc[x], a, b[2 * x], b[2 * x + 1]);
                mma_bf16_16816(acc[x], a, c[2 * x], c[2 * x + 1]);
                mma_bf16_16816(acc[x], a2, b[2 * x], b[2 * x + 1]);
            }
        }
        bf16* ug = dp.u + at * 2 * CT * dv + j0;
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = u ? r1 : r0, j = (half * 2 + x) * 8 + c4 * 2;
                uint32_t wh, wl;
                split_bf162(u0[x][u].x - acc[x][u * 2], u0[x][u].y - acc[x][u * 2 + 1], wh, wl);
                *reinterpret_cast<uint32_t*>(uh + r * LDS + j) = wh;
                *reinterpret_cast<uint32_t*>(ul + r * LDS + j) = wl;
                if (half * 2 + x < nn) {
                    *reinterpret_cast<uint32_t*>(ug + (size_t)r * dv + j) = wh;
                    *reinterpret_cast<uint32_t*>(ug + (size_t)(CT + r) * dv + j) = wl;
                }
            }
        __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int row = (warp + m * 8) * 16;
            if (row >= dkp) continue;
            const float k0 = exp2f(keep[m][0]), k1 = exp2f(keep[m][1]);
#pragma unroll
            for (int x = 0; x < 4; ++x) { S[m][x][0] *= k0; S[m][x][1] *= k0; S[m][x][2] *= k1; S[m][x][3] *= k1; }
#pragma unroll
            for (int ks = 0; ks < CT; ks += 16) {
                const int off = (ks + (lane & 7) + ((lane >> 4) & 1) * 8) * ldk + row + ((lane >> 3) & 1) * 8;
                uint32_t a[4], a2[4];
                ldsm_x4_trans(a, kt + off);
                ldsm_x4_trans(a2, kt + tile + off);
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    uint32_t b[4], c[4];
                    ldsm_x4_trans(b, uh + (ks + (lane & 15)) * LDS + x * 16 + (lane >> 4) * 8);
                    ldsm_x4_trans(c, ul + (ks + (lane & 15)) * LDS + x * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int y = 0; y < 2; ++y) {
                        mma_bf16_16816(S[m][x * 2 + y], a, b[2 * y], b[2 * y + 1]);
                        mma_bf16_16816(S[m][x * 2 + y], a, c[2 * y], c[2 * y + 1]);
                        mma_bf16_16816(S[m][x * 2 + y], a2, b[2 * y], b[2 * y + 1]);
                    }
                }
            }
        }
        __syncthreads();
        if (dp.stages == 1) fetch(i + 1);
    }
    cp_async_wait_all();
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int r = (warp + m * 8) * 16 + g + u * 8;
                if (r < dk && i < nn) *reinterpret_cast<float2*>(state + (size_t)r * dv + i * 8 + c4 * 2) = make_float2(S[m][i][u * 2], S[m][i][u * 2 + 1]);
            }
}

}  // namespace

// 1 when the chunked kernels take these sizes (head rows of whole 16-byte pieces, tiles that fit in shared memory).
SL_API int sl_delta_chunk_ok(int dk, int dv) {
    if (dk < 8 || dv < 8 || dk % 8 != 0 || dv % 8 != 0 || dk > 256 || dv > 256) return 0;
    int slab, bufs;
    return prepare_smem(dk, dv) <= SMEM_MAX && scan_smem(dk, 1) <= SMEM_MAX && plan_output(KIND_DELTA, dk, dv, slab, bufs) <= SMEM_MAX;
}

// One pass over the chunks [c0, c1) of B sequences (bf16 rows in and out).  Passes of one step run in order on one stream.
SL_API int sl_delta_chunks(const DeltaChunkParams* args, int B, cudaStream_t s) {
    DeltaChunkParams params = *args;
    DeltaChunkParams* p = &params;
    GatedScanParams& sp = p->c.s;
    if (B == 0 || p->c.c1 <= p->c.c0) return 0;
    if (!sl_delta_chunk_ok(sp.dk, sp.dv) || sp.ld % 8 != 0 || sp.ldg % 2 != 0 || sp.ldo % 2 != 0 || sp.group < 1 || B > 65535 || sp.h > 65535) return -1;
    if (((uintptr_t)sp.q | (uintptr_t)sp.k | (uintptr_t)sp.v) % 16 != 0 || ((uintptr_t)sp.g | (uintptr_t)sp.out) % 4 != 0) return -1;
    const int dk = sp.dk, dv = sp.dv, h = sp.h, nc = p->c.c1 - p->c.c0;
    const size_t s1 = prepare_smem(dk, dv), s3 = plan_output(KIND_DELTA, dk, dv, p->c.slab, p->c.slab_bufs);
    p->stages = scan_smem(dk, 2) <= SMEM_MAX ? 2 : 1;
    const size_t s2 = scan_smem(dk, p->stages);
#define SL_RUN(KERN, GRID, THREADS, BYTES, ARG)                                                                    \
    {                                                                                                              \
        auto kern = KERN;                                                                                          \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(BYTES));                     \
        sl_launch(kern, GRID, THREADS, BYTES, s, ARG);                                                             \
    }
    if (dk <= 128) SL_RUN(delta_prepare_kernel<16>, dim3(nc, h), 256, s1, *p)
    else SL_RUN(delta_prepare_kernel<32>, dim3(nc, h), 256, s1, *p)
    const dim3 grid((dv + NV - 1) / NV, h, B);
    if (dk <= 128) SL_RUN(delta_scan_kernel<1>, grid, 256, s2, *p)
    else SL_RUN(delta_scan_kernel<2>, grid, 256, s2, *p)
    p->c.u = p->u;
    p->c.unit = p->unit;
    if (dv <= 128) SL_RUN((chunk_output_kernel<KIND_DELTA, 4>), dim3(nc, h), OUT_THREADS, s3, p->c)
    else SL_RUN((chunk_output_kernel<KIND_DELTA, 8>), dim3(nc, h), OUT_THREADS, s3, p->c)
#undef SL_RUN
    return SL_LAUNCH_CHECK();
}
