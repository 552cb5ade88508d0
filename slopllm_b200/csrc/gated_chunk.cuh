// Parts of the chunked recurrences that the kinds share: parameters, row loads and the output kernel (see gated_chunk.cu for GLA
// and mLSTM, delta_chunk.cu for the gated delta rule).
#pragma once

#include "gated_scan.cuh"
#include "mma_sync.cuh"

namespace {

constexpr int CT = 64;                       // tokens per chunk

struct GatedChunkParams {
    GatedScanParams s;
    const int* chunks;                       // [chunks][4]: sequence, first token, tokens, 1 if the sequence's last chunk
    const int* seq_chunks;                   // [B + 1]
    int c0, c1;                              // chunk range of this pass
    float* b;                                // GLA, delta: running log2 decays [T, h * dk]
    float* loc;                              // [chunks of the pass, h, dk, dv]: own contribution, then S_in: eight high bf16 terms,
                                             // then their eight low terms, in the place of every eight values
    float* nloc;                             // mLSTM: [chunks of the pass, h, dk], then n_in
    float* scal;                             // mLSTM: [chunks of the pass, h, 4]: b_C, M_C, m_in, m after the chunk
    const bf16* u;                           // delta: the updates in the place of v, [chunks of the pass, h, high | low, CT, dv]
    const float* unit;                       // delta: factors that make q (with dk^-0.5) and k unit vectors, [T, h, 2]
    int slab, slab_bufs;                     // set by the launcher: state rows per slab, slabs in shared memory at a time (1 or 2)
};

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

// One warp: a_s = i_s - b_s, b_s, and the running maximum M_s of a over the chunk's tokens (two tokens per lane).
__device__ __forceinline__ void mlstm_gates(const GatedScanParams& p, int t0, int n, int h, float* a_s, float* b_s, float* mx_s) {
    const int lane = threadIdx.x & 31;
    float gi[2], gf[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int s = lane * 2 + j;
        gi[j] = -INFINITY;
        gf[j] = 0.f;
        if (s < n) {
            const float* gr = p.gates + (size_t)(t0 + s) * p.ld_gates;
            gi[j] = p.cap * tanhf((gr[h] + p.i_b[h]) / p.cap);
            gf[j] = logsigmoid_f(p.cap * tanhf((gr[p.h + h] + p.f_b[h]) / p.cap));
        }
    }
    float sum = gf[0] + gf[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += x;
    }
    float before = __shfl_up_sync(0xffffffffu, sum, 1);
    if (lane == 0) before = 0.f;
    const float b0 = before + gf[0], b1 = b0 + gf[1];
    const float a0 = gi[0] - b0, a1 = gi[1] - b1;
    float mx = fmaxf(a0, a1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, x);
    }
    float mb = __shfl_up_sync(0xffffffffu, mx, 1);
    if (lane == 0) mb = -INFINITY;
    a_s[lane * 2] = a0; a_s[lane * 2 + 1] = a1;
    b_s[lane * 2] = b0; b_s[lane * 2 + 1] = b1;
    mx_s[lane * 2] = fmaxf(mb, a0); mx_s[lane * 2 + 1] = fmaxf(fmaxf(mb, a0), a1);
}

// ---- outputs -----------------------------------------------------------------------------------------------------------------
constexpr int OUT_THREADS = 512;             // 16 warps: 4 row tiles of 16 tokens x 4 column quarters
constexpr int LDA = CT + 8;

size_t output_smem(int kind, int dk, int dv, int slab, int bufs) {
    const int dkp = (dk + 15) / 16 * 16;
    const size_t slabs = (size_t)bufs * 2 * slab * (dv + 8) * 2, scores = (size_t)2 * CT * LDA * 2;
    size_t b = (size_t)CT * (dkp + 8) * 2 * 2 + (size_t)CT * (dv + 8) * 2 * (kind == KIND_DELTA ? 2 : 1) + (slabs > scores ? slabs : scores);
    b += kind != KIND_MLSTM ? (size_t)CT * (dkp + 4) * 4 : 0;
    return b + (size_t)CT * 12 * 4;
}
constexpr size_t SMEM_MAX = 220 * 1024, SMEM_TWO = 112 * 1024;       // one block per SM, two

// Slabs that let two blocks share an SM where possible, then as much of the state as fits.  Returns the bytes.
size_t plan_output(int kind, int dk, int dv, int& slab, int& bufs) {
    const int plans[][2] = {{64, 2}, {64, 1}, {32, 2}, {32, 1}, {16, 1}};
    for (size_t limit : {SMEM_TWO, SMEM_MAX})
        for (auto& pl : plans) {
            slab = pl[0];
            bufs = pl[1];
            const size_t b = output_smem(kind, dk, dv, slab, bufs);
            if (b <= limit && (bufs == 1 || dk > slab)) return b;
        }
    return SMEM_MAX + 1;
}

// grid (chunks of the pass, h).  NT: 8-wide value tiles per column quarter (dv <= 32 * NT).
template <int KIND, int NT>
__global__ void __launch_bounds__(OUT_THREADS, NT <= 4 ? 2 : 1) chunk_output_kernel(GatedChunkParams cp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    constexpr bool DECAY = KIND != KIND_MLSTM, DELTA = KIND == KIND_DELTA;
    const GatedScanParams& p = cp.s;
    const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int rt = warp & 3, quarter = warp >> 2, hq = h / p.group;
    const int* ch = cp.chunks + (size_t)(cp.c0 + ci) * 4;
    const int seq = ch[0], t0 = ch[1], n = ch[2], last = ch[3], dk = p.dk, dv = p.dv;
    const int dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8, ldb = dkp + 4;
    bf16* qs = reinterpret_cast<bf16*>(smraw);           // [CT][ldk]
    bf16* ks = qs + CT * ldk;
    bf16* vs = ks + CT * ldk;                            // [CT][ldv]
    bf16* slabs = vs + (DELTA ? 2 : 1) * CT * ldv;       // (delta: the low terms of v follow) state rows [slab][ldv], high and low terms, one or two slabs; then
    bf16* ah = slabs;                                    // [CT][LDA] scores, high and low terms
    bf16* al = ah + CT * LDA;
    const int slab = cp.slab, region = max(cp.slab_bufs * 2 * slab * ldv, 2 * CT * LDA);
    float* fs = reinterpret_cast<float*>(slabs + region);
    float* bs = fs;                                      // GLA: [CT][ldb]
    float* rows = fs + (DECAY ? CT * ldb : 0);
    float *ga = rows, *gb = rows + CT, *gx = rows + 2 * CT, *qn = rows + 3 * CT, *nq = rows + 4 * CT, *ssq = rows + 8 * CT;
    const float qscale = rsqrtf((float)dk);
    const size_t base = (size_t)ci * p.h + h;
    const bf16* sin = reinterpret_cast<const bf16*>(cp.loc + base * dk * dv);
    auto load_slab = [&](int k0) {
        bf16* sh = slabs + (k0 / slab) % cp.slab_bufs * 2 * slab * ldv;
        const int per = dv / 8, rowsn = min(slab, dkp - k0);
        for (int i = tid; i < rowsn * per; i += OUT_THREADS) {
            const int r = i / per, c = i % per;
            bf16* dst = sh + r * ldv + c * 8;
            if (k0 + r < dk) {
                const bf16* src = sin + ((size_t)(k0 + r) * dv + c * 8) * 2;
                cp_async16(dst, src);
                cp_async16(dst + slab * ldv, src + 8);
            } else {
                *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<uint4*>(dst + slab * ldv) = make_uint4(0, 0, 0, 0);
            }
        }
    };
    load_rows(qs, ldk, (const bf16*)p.q + (size_t)t0 * p.ld + hq * dk, p.ld, n, dk, dkp);
    if (DECAY) {
        const int per = dkp / 4;
        for (int i = tid; i < CT * per; i += OUT_THREADS) {
            const int s = i / per, c = (i % per) * 4;
            if (s < n && c < dk) cp_async16(bs + s * ldb + c, cp.b + (size_t)(t0 + s) * (p.h * dk) + h * dk + c);
            else *reinterpret_cast<float4*>(bs + s * ldb + c) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    load_slab(0);
    if (cp.slab_bufs > 1) load_slab(slab);
    cp_async_commit();
    load_rows(ks, ldk, (const bf16*)p.k + (size_t)t0 * p.ld + hq * dk, p.ld, n, dk, dkp);
    if (DELTA) {
        load_rows(vs, ldv, cp.u + base * 2 * CT * dv, dv, CT, dv, dv);
        load_rows(vs + CT * ldv, ldv, cp.u + (base * 2 + 1) * CT * dv, dv, CT, dv, dv);
        if (tid < CT) {
            const float2 f = tid < n ? *reinterpret_cast<const float2*>(cp.unit + ((size_t)(t0 + tid) * p.h + h) * 2) : make_float2(0.f, 0.f);
            ga[tid] = f.y;
            gb[tid] = f.x;
        }
    } else {
        load_rows(vs, ldv, (const bf16*)p.v + (size_t)t0 * p.ld + h * dv, p.ld, n, dv, dv);
    }
    cp_async_commit();
    const float m_in = KIND == KIND_MLSTM ? cp.scal[base * 4 + 2] : 0.f;
    if (KIND == KIND_MLSTM && warp == 0) mlstm_gates(p, t0, n, h, ga, gb, gx);
    cp_async_wait<1>();
    __syncthreads();
    if (KIND == KIND_MLSTM) {
        if (tid < CT) gx[tid] = fmaxf(gx[tid], m_in);
        // q_t . n_in: eight lanes per token
        float a = 0.f;
        const float* nin = cp.nloc + base * dk;
        const int r = tid >> 3;
        for (int c = tid & 7; c < dk; c += 8) a += __bfloat162float(qs[r * ldk + c]) * nin[c];
#pragma unroll
        for (int o = 1; o < 8; o <<= 1) a += __shfl_xor_sync(0xffffffffu, a, o);
        if ((tid & 7) == 0) qn[r] = a;
        __syncthreads();
    }
    // ---- S_in part: rows of the state in slabs ----
    const int ntiles = dv / 8, tq = (ntiles + 3) / 4, nt0 = quarter * tq, ntn = max(0, min(tq, ntiles - nt0));
    const int r0 = rt * 16 + g, r1 = r0 + 8;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int k0 = 0; k0 < dkp; k0 += slab) {
        const int rowsn = min(slab, dkp - k0);
        const bf16* sh = slabs + (k0 / slab) % cp.slab_bufs * 2 * slab * ldv;
        const bf16* sl = sh + slab * ldv;
        if (k0 >= cp.slab_bufs * slab) {                             // further slabs take the buffers in turn
            cp_async_wait<0>();
            __syncthreads();
        }
        for (int kk = 0; kk < rowsn; kk += 16) {
            uint32_t a[4], a2[4];
            if (KIND == KIND_MLSTM) {
                ldsm_x4(a, qs + (rt * 16 + (lane & 15)) * ldk + k0 + kk + (lane >> 4) * 8);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int r = (i & 1) ? r1 : r0, c = k0 + kk + c4 * 2 + (i >> 1) * 8;
                    const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                    const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c);
                    const float f = DELTA ? gb[r] : qscale;
                    split_bf162(x.x * f * exp2_fast(b.x), x.y * f * exp2_fast(b.y), a[i], a2[i]);
                }
            }
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                if (i >= ntn) break;
                uint32_t b0, b1, l0, l1;
                ldsm_x2_trans(b0, b1, sh + (kk + (lane & 15)) * ldv + (nt0 + i) * 8);
                ldsm_x2_trans(l0, l1, sl + (kk + (lane & 15)) * ldv + (nt0 + i) * 8);
                mma_bf16_16816(acc[i], a, b0, b1);
                mma_bf16_16816(acc[i], a, l0, l1);
                if (DECAY) mma_bf16_16816(acc[i], a2, b0, b1);
            }
        }
        if (k0 + cp.slab_bufs * slab < dkp) {
            __syncthreads();
            load_slab(k0 + cp.slab_bufs * slab);
            cp_async_commit();
        }
    }
    float e0 = 1.f, e1 = 1.f;
    if (KIND == KIND_MLSTM) {
        e0 = __expf(m_in - gx[r0]) * qscale;
        e1 = __expf(m_in - gx[r1]) * qscale;
#pragma unroll
        for (int i = 0; i < NT; ++i) { acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1; }
    }
    cp_async_wait<0>();
    __syncthreads();                                     // (the scores take the place of the state slabs)
    // ---- scores of (row tile rt, key tile J = quarter) ----
    {
        const int J = quarter, r0 = rt * 16 + g, r1 = r0 + 8;
        float sc[2][4] = {};
        if (KIND == KIND_MLSTM ? J <= rt : J < rt) {
            for (int kk = 0; kk < dkp; kk += 16) {
                uint32_t a[4], a2[4];
                if (KIND == KIND_MLSTM) {
                    ldsm_x4(a, qs + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
                } else {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int r = (i & 1) ? r1 : r0, c = kk + c4 * 2 + (i >> 1) * 8;
                        const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                        const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c);
                        const float2 an = *reinterpret_cast<const float2*>(bs + (rt * 16 - 1) * ldb + c);
                        split_bf162(x.x * exp2_fast(fminf(b.x - an.x, 0.f)), x.y * exp2_fast(fminf(b.y - an.y, 0.f)), a[i], a2[i]);
                    }
                }
#pragma unroll
                for (int t = 0; t < 2; ++t) {
                    const int s = J * 16 + t * 8;
                    if (KIND == KIND_MLSTM) {
                        uint32_t b0, b1;
                        ldsm_x2(b0, b1, ks + (s + (lane & 7)) * ldk + kk + ((lane >> 3) & 1) * 8);
                        mma_bf16_16816(sc[t], a, b0, b1);
                    } else {
                        uint32_t bh[2], bl[2];
#pragma unroll
                        for (int i = 0; i < 2; ++i) {
                            const int c = kk + c4 * 2 + i * 8;
                            const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + (s + g) * ldk + c));
                            const float2 b = *reinterpret_cast<const float2*>(bs + (s + g) * ldb + c);
                            const float2 an = *reinterpret_cast<const float2*>(bs + (rt * 16 - 1) * ldb + c);
                            split_bf162(x.x * exp2_fast(fminf(an.x - b.x, 0.f)), x.y * exp2_fast(fminf(an.y - b.y, 0.f)), bh[i], bl[i]);
                        }
                        mma_bf16_16816(sc[t], a, bh[0], bh[1]);
                        mma_bf16_16816(sc[t], a, bl[0], bl[1]);
                        mma_bf16_16816(sc[t], a2, bh[0], bh[1]);
                    }
                }
            }
        }
        if (KIND == KIND_MLSTM || J != rt) {
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                float v[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int r = i < 2 ? r0 : r1, s = J * 16 + t * 8 + c4 * 2 + (i & 1);
                    float w = DELTA ? gb[r] * ga[s] : qscale;
                    if (KIND == KIND_MLSTM) w *= s < n ? __expf(ga[s] - gx[r]) : 0.f;
                    v[i] = s <= r ? sc[t][i] * w : 0.f;
                }
                sum0 += v[0] + v[1];
                sum1 += v[2] + v[3];
                uint32_t hi, lo;
                const int s = J * 16 + t * 8 + c4 * 2;
                split_bf162(v[0], v[1], hi, lo);
                *reinterpret_cast<uint32_t*>(ah + r0 * LDA + s) = hi;
                *reinterpret_cast<uint32_t*>(al + r0 * LDA + s) = lo;
                split_bf162(v[2], v[3], hi, lo);
                *reinterpret_cast<uint32_t*>(ah + r1 * LDA + s) = hi;
                *reinterpret_cast<uint32_t*>(al + r1 * LDA + s) = lo;
            }
            if (KIND == KIND_MLSTM) {
                sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1); sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
                sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1); sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
                if (c4 == 0) { nq[r0 * 4 + J] = sum0; nq[r1 * 4 + J] = sum1; }
            }
        }
    }
    if (DECAY) {
        // diagonal blocks: the 136 pairs s <= r of each, a quad of lanes per pair, channel pairs interleaved over the quad
        for (int it = tid >> 2; it < 4 * 136; it += OUT_THREADS / 4) {
            const int blk = it / 136, x = it % 136, i = x / 17, j = x % 17;          // rows i and 15 - i together have 17 pairs
            const int r = blk * 16 + (j <= i ? i : 15 - i), s = blk * 16 + (j <= i ? j : j - i - 1);
            float a0 = 0.f, a1 = 0.f;
            if (r < n) {
#pragma unroll 4
                for (int c = (tid & 3) * 2; c < dk; c += 8) {
                    const float2 qv = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                    const float2 kv = bf162_to_f2(*reinterpret_cast<const uint32_t*>(ks + s * ldk + c));
                    const float2 br = *reinterpret_cast<const float2*>(bs + r * ldb + c), b2 = *reinterpret_cast<const float2*>(bs + s * ldb + c);
                    a0 += qv.x * kv.x * exp2_fast(br.x - b2.x);
                    a1 += qv.y * kv.y * exp2_fast(br.y - b2.y);
                }
            }
            float a = a0 + a1;
            a += __shfl_xor_sync(0xffffffffu, a, 1);
            a += __shfl_xor_sync(0xffffffffu, a, 2);
            if ((tid & 3) == 0) {
                a *= DELTA ? gb[r] * ga[s] : qscale;
                const bf16 hi = __float2bfloat16(a);
                ah[r * LDA + s] = hi;
                al[r * LDA + s] = __float2bfloat16(a - __bfloat162float(hi));
                if (s != r) ah[s * LDA + r] = al[s * LDA + r] = __float2bfloat16(0.f);
            }
        }
    }
    __syncthreads();
    // ---- intra-chunk part ----
    for (int kk = 0; kk <= rt * 16; kk += 16) {
        uint32_t a[4], a2[4];
        ldsm_x4(a, ah + (rt * 16 + (lane & 15)) * LDA + kk + (lane >> 4) * 8);
        ldsm_x4(a2, al + (rt * 16 + (lane & 15)) * LDA + kk + (lane >> 4) * 8);
#pragma unroll
        for (int i = 0; i < NT; ++i) {
            if (i >= ntn) break;
            uint32_t b0, b1;
            ldsm_x2_trans(b0, b1, vs + (kk + (lane & 15)) * ldv + (nt0 + i) * 8);
            mma_bf16_16816(acc[i], a, b0, b1);
            mma_bf16_16816(acc[i], a2, b0, b1);
            if (DELTA) {
                ldsm_x2_trans(b0, b1, vs + CT * ldv + (kk + (lane & 15)) * ldv + (nt0 + i) * 8);
                mma_bf16_16816(acc[i], a, b0, b1);
            }
        }
    }
    if (KIND == KIND_MLSTM) {
        const float q0 = e0 * qn[r0] + nq[r0 * 4] + nq[r0 * 4 + 1] + nq[r0 * 4 + 2] + nq[r0 * 4 + 3];
        const float q1 = e1 * qn[r1] + nq[r1 * 4] + nq[r1 * 4 + 1] + nq[r1 * 4 + 2] + nq[r1 * 4 + 3];
        const float d0 = 1.f / (fmaxf(fabsf(q0), expf(-(gb[r0] + gx[r0]))) + 1e-6f), d1 = 1.f / (fmaxf(fabsf(q1), expf(-(gb[r1] + gx[r1]))) + 1e-6f);
#pragma unroll
        for (int i = 0; i < NT; ++i) { acc[i][0] *= d0; acc[i][1] *= d0; acc[i][2] *= d1; acc[i][3] *= d1; }
        if ((last || cp.c0 + ci + 1 == cp.c1) && tid == 0) p.m[(size_t)p.state_idx[seq] * p.h + h] = cp.scal[base * 4 + 3];
    }
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
    const float* nw = p.norm_w + (KIND == KIND_MLSTM ? (size_t)h * dv : 0);
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        if (i >= ntn) break;
        const int j = (nt0 + i) * 8 + c4 * 2;
        const float2 w = make_float2(nw[j], nw[j + 1]);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = u ? r1 : r0;
            if (r >= n) continue;
            const float inv = u ? i1 : i0;
            const float2 gt = bf162_to_f2(*reinterpret_cast<const uint32_t*>((const bf16*)p.g + (size_t)(t0 + r) * p.ldg + h * dv + j));
            const float x = 1.f / (1.f + __expf(-gt.x)), y = 1.f / (1.f + __expf(-gt.y));
            const float gx0 = KIND == KIND_GLA ? gt.x * x : x, gy0 = KIND == KIND_GLA ? gt.y * y : y;
            *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)(t0 + r) * p.ldo + (size_t)h * dv + j) =
                f2_to_bf162(acc[i][u * 2] * inv * w.x * gx0, acc[i][u * 2 + 1] * inv * w.y * gy0);
        }
    }
}

}  // namespace
