// Chunked form of the gated outer-product recurrences (see gated_scan.cu) for portions of prompts, on the tensor cores.
//
// A sequence's tokens are cut into chunks of 64.  With b_t the running sum of the log decay inside a chunk,
//
//   GLA    o_t = (q_t e^{b_t}) . S_in + sum_{s<=t} [sum_c q_t[c] k_s[c] e^{b_t[c] - b_s[c]}] v_s
//          S_out = diag(e^{b_C}) S_in + sum_s (k_s e^{b_C - b_s}) v_s^T
//   mLSTM  with a_s = i_s - b_s, M_t = max_{s<=t} a_s, x_t = max(m_in, M_t), m_t = b_t + x_t:
//          S_t^T q_t = e^{m_in - x_t} S_in^T q_t + sum_{s<=t} e^{a_s - x_t} (q_t . k_s) v_s   (n_t . q_t likewise without v)
//          S_out = e^{m_in - x_C} S_in + e^{M_C - x_C} sum_s (k_s e^{a_s - M_C}) v_s^T
//
//   retention  with t, s the places inside the chunk, gamma the head's decay, q and k turned by their positions:
//          o_t = gamma^{t+1} q_t . S_in + sum_{s<=t} gamma^{t-s} (q_t . k_s) v_s
//          S_out = gamma^C S_in + sum_s (k_s gamma^{C-1-s}) v_s^T
//
// in three launches:
//   1 chunk_state_kernel   (chunk, head): decays, the chunk's own state contribution
//   2 chunk_scan_kernel    (elements, head, sequence): carries the fp32 state over the chunks and leaves each chunk's S_in
//   3 chunk_output_kernel  (chunk, head): intra-chunk and S_in parts, normaliser, head norm, output gate
//
// No exponent is ever positive: the products e^{b_t - b_s} of GLA are taken directly inside 16-token diagonal blocks and
// through an anchor between the blocks otherwise.  q, k, v come as bf16; every other operand of a tensor-core product (decayed
// keys and queries, turned ones, scores, the state) is split into two bf16 terms, so the results keep fp32-like accuracy.
#include "gated_chunk.cuh"

namespace {

struct GatedChunkParams {
    GatedScanParams s;
    const int* chunks;                       // [chunks][4]: sequence, first token, tokens, 1 if the sequence's last chunk
    const int* seq_chunks;                   // [B + 1]
    int c0, c1;                              // chunk range of this pass
    float* b;                                // GLA: running log2 decays [T, h * dk]
    float* loc;                              // [chunks of the pass, h, dk, dv]: own contribution, then S_in: eight high bf16 terms,
                                             // then their eight low terms, in the place of every eight values
    float* nloc;                             // mLSTM: [chunks of the pass, h, dk], then n_in
    float* scal;                             // mLSTM: [chunks of the pass, h, 4]: b_C, M_C, m_in, m after the chunk
    int slab, slab_bufs;                     // set by the launcher: state rows per slab, slabs in shared memory at a time (1 or 2)
};

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

// ---- 1: decays and the chunk's own state contribution -----------------------------------------------------------------------
// grid (chunks of the pass, h), block 256
template <int KIND>
__global__ void __launch_bounds__(256) chunk_state_kernel(GatedChunkParams cp) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const GatedScanParams& p = cp.s;
    const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int* ch = cp.chunks + (size_t)(cp.c0 + ci) * 4;
    const int t0 = ch[1], n = ch[2], dk = p.dk, dv = p.dv;
    const int dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8;
    bf16* kh = reinterpret_cast<bf16*>(smraw);           // [CT][ldk] keys, then decayed keys: high and low terms
    bf16* kl = kh + CT * ldk;
    bf16* vs = kl + CT * ldk;                            // [CT][ldv]
    float* fs = reinterpret_cast<float*>(vs + CT * ldv); // GLA: log2 decays [CT][dk], then the inputs; mLSTM: a, b, M
    load_rows(kh, ldk, (const bf16*)p.k + (size_t)t0 * p.ld + h * dk, p.ld, n, dk, dkp);
    load_rows(vs, ldv, (const bf16*)p.v + (size_t)t0 * p.ld + h * dv, p.ld, n, dv, dv);
    cp_async_commit();
    if (KIND == KIND_GLA) {
        float* low = fs + CT * dk;                       // [CT][rank]
        bf16* a2 = reinterpret_cast<bf16*>(low + CT * p.rank);       // [dk][rank]
        const bf16* a2g = (const bf16*)p.a2 + (size_t)h * dk * p.rank;
#pragma unroll 4
        for (int i = tid; i < dk * p.rank; i += 256) a2[i] = a2g[i];
#pragma unroll 4
        for (int i = tid; i < CT * p.rank; i += 256)
            low[i] = i < n * p.rank ? p.gates[(size_t)(t0 + i / p.rank) * p.ld_gates + i % p.rank] : 0.f;
        __syncthreads();
        for (int i = tid; i < dk * (CT / 8); i += 256) {                 // a channel, eight tokens
            const int c = i % dk, s0 = i / dk * 8;
            if (s0 >= n) continue;
            float z[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) z[j] = p.a2_b[h * dk + c];
#pragma unroll 4
            for (int r = 0; r < p.rank; ++r) {
                const float w = __bfloat162float(a2[c * p.rank + r]);
#pragma unroll
                for (int j = 0; j < 8; ++j) z[j] += w * low[(s0 + j) * p.rank + r];
            }
            const float scale = p.inv_tau * LOG2E;
#pragma unroll
            for (int j = 0; j < 8; ++j) fs[(s0 + j) * dk + c] = logsigmoid_f(z[j]) * scale;
        }
        __syncthreads();
        for (int c = tid; c < dk; c += 256) {
            float run = 0.f;
#pragma unroll 8
            for (int s = 0; s < n; ++s) {
                run += fs[s * dk + c];
                fs[s * dk + c] = run;
            }
        }
        __syncthreads();
        for (int i = tid; i < n * (dk / 4); i += 256) {
            const int s = i / (dk / 4), c = (i % (dk / 4)) * 4;
            *reinterpret_cast<float4*>(cp.b + (size_t)(t0 + s) * (p.h * dk) + h * dk + c) = *reinterpret_cast<const float4*>(fs + s * dk + c);
        }
    } else if (KIND == KIND_MLSTM && warp == 0) {
        mlstm_gates(p, t0, n, h, fs, fs + CT, fs + 2 * CT);
    }
    cp_async_wait<0>();
    __syncthreads();
    const float top = KIND == KIND_MLSTM ? fs[2 * CT + n - 1] : 0.f, rate = KIND == KIND_RETENTION ? p.decay[p.h + h] : 0.f;
    for (int i = tid; i < CT * (dkp / 2); i += 256) {
        const int s = i / (dkp / 2), c = (i % (dkp / 2)) * 2;
        uint32_t hi = 0, lo = 0;
        if (s < n && c < dk) {
            float2 k = bf162_to_f2(*reinterpret_cast<const uint32_t*>(kh + s * ldk + c));
            if (KIND == KIND_RETENTION) k = turned(p, t0 + s, c, k);
            float w0, w1;
            if (KIND == KIND_GLA) {
                w0 = exp2_fast(fs[(n - 1) * dk + c] - fs[s * dk + c]);
                w1 = exp2_fast(fs[(n - 1) * dk + c + 1] - fs[s * dk + c + 1]);
            } else if (KIND == KIND_MLSTM) {
                w0 = w1 = __expf(fs[s] - top);
            } else {
                w0 = w1 = exp2f((float)(n - 1 - s) * rate);
            }
            split_bf162(k.x * w0, k.y * w1, hi, lo);
        }
        *reinterpret_cast<uint32_t*>(kh + s * ldk + c) = hi;
        *reinterpret_cast<uint32_t*>(kl + s * ldk + c) = lo;
    }
    __syncthreads();
    const size_t base = (size_t)ci * p.h + h;
    if (KIND == KIND_MLSTM) {
        for (int c = tid; c < dk; c += 256) {
            float a = 0.f;
#pragma unroll 8
            for (int s = 0; s < n; ++s) a += __bfloat162float(kh[s * ldk + c]) + __bfloat162float(kl[s * ldk + c]);
            cp.nloc[base * dk + c] = a;
        }
        if (tid == 0) { cp.scal[base * 4] = fs[CT + n - 1]; cp.scal[base * 4 + 1] = top; }
    }
    // loc[c, j] = sum_s k~[s, c] v[s, j]: units of 16 channels x 64 values over the warps
    float* loc = cp.loc + base * dk * dv;
    const int cols = (dv + 63) / 64, units = dkp / 16 * cols, ksteps = (n + 15) / 16, g = lane >> 2, q = lane & 3;
    for (int u = warp; u < units; u += 8) {
        const int m0 = u / cols * 16, j0 = u % cols * 64, nt = min(8, (dv - j0) / 8);
        float acc[8][4] = {};
        for (int ks = 0; ks < ksteps; ++ks) {
            const int off = (ks * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * ldk + m0 + ((lane >> 3) & 1) * 8;
            uint32_t ah[4], al[4];
            ldsm_x4_trans(ah, kh + off);
            ldsm_x4_trans(al, kl + off);
#pragma unroll
            for (int i = 0; i < 8; ++i) {
                if (i >= nt) break;
                uint32_t b0, b1;
                ldsm_x2_trans(b0, b1, vs + (ks * 16 + (lane & 15)) * ldv + j0 + i * 8);
                mma_bf16_16816(acc[i], ah, b0, b1);
                mma_bf16_16816(acc[i], al, b0, b1);
            }
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (i >= nt) break;
            const int j = j0 + i * 8 + q * 2;
            if (m0 + g < dk) *reinterpret_cast<float2*>(loc + (size_t)(m0 + g) * dv + j) = make_float2(acc[i][0], acc[i][1]);
            if (m0 + g + 8 < dk) *reinterpret_cast<float2*>(loc + (size_t)(m0 + g + 8) * dv + j) = make_float2(acc[i][2], acc[i][3]);
        }
    }
}

// ---- 2: the state over the chunks --------------------------------------------------------------------------------------------
// grid (ceil(dk * dv / 2048), h, B), block 256: eight consecutive values of a state row per thread
template <int KIND>
__global__ void __launch_bounds__(256) chunk_scan_kernel(GatedChunkParams cp) {
    pdl_grid_sync();
    const GatedScanParams& p = cp.s;
    const int h = blockIdx.y, seq = blockIdx.z, dk = p.dk, dv = p.dv;
    const int lo = max(cp.seq_chunks[seq], cp.c0), hi = min(cp.seq_chunks[seq + 1], cp.c1);
    if (lo >= hi) return;
    const size_t slot = (size_t)p.state_idx[seq] * p.h + h, size = (size_t)dk * dv;
    const int e = (blockIdx.x * 256 + threadIdx.x) * 8;
    const float m0 = KIND == KIND_MLSTM ? p.m[slot] : 0.f;
    if (e < (int)size) {
        const int c = e / dv;
        float S[8];
        *reinterpret_cast<float4*>(S) = *reinterpret_cast<const float4*>(p.S + slot * size + e);
        *reinterpret_cast<float4*>(S + 4) = *reinterpret_cast<const float4*>(p.S + slot * size + e + 4);
        float m = m0;
        constexpr int U = 4;                              // chunks whose contributions are in flight
        for (int i0 = lo; i0 < hi; i0 += U) {
            float x[U][8], d[U], bc[U];                   // (mLSTM: d = M_C, bc = b_C)
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const int i = min(i0 + j, hi - 1);
                const float* src = cp.loc + ((size_t)(i - cp.c0) * p.h + h) * size + e;
                *reinterpret_cast<float4*>(x[j]) = *reinterpret_cast<const float4*>(src);
                *reinterpret_cast<float4*>(x[j] + 4) = *reinterpret_cast<const float4*>(src + 4);
                if (KIND == KIND_MLSTM) {
                    bc[j] = cp.scal[((size_t)(i - cp.c0) * p.h + h) * 4];
                    d[j] = cp.scal[((size_t)(i - cp.c0) * p.h + h) * 4 + 1];
                } else {
                    const int* ch = cp.chunks + (size_t)i * 4;
                    d[j] = KIND == KIND_RETENTION ? (float)ch[2] * p.decay[p.h + h] : cp.b[(size_t)(ch[1] + ch[2] - 1) * (p.h * dk) + h * dk + c];
                }
            }
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const int i = i0 + j;
                if (i >= hi) break;
                float add = 1.f, keep = KIND == KIND_MLSTM ? 1.f : exp2f(d[j]);
                if (KIND == KIND_MLSTM) {
                    const float top = fmaxf(m, d[j]);
                    keep = expf(m - top);
                    add = expf(d[j] - top);
                    m = bc[j] + top;
                }
                uint4 wh, wl;
                split_bf162(S[0], S[1], wh.x, wl.x); split_bf162(S[2], S[3], wh.y, wl.y);
                split_bf162(S[4], S[5], wh.z, wl.z); split_bf162(S[6], S[7], wh.w, wl.w);
                uint4* dst = reinterpret_cast<uint4*>(cp.loc + ((size_t)(i - cp.c0) * p.h + h) * size + e);
                dst[0] = wh;
                dst[1] = wl;
#pragma unroll
                for (int y = 0; y < 8; ++y) S[y] = keep * S[y] + add * x[j][y];
            }
        }
        *reinterpret_cast<float4*>(p.S + slot * size + e) = *reinterpret_cast<const float4*>(S);
        *reinterpret_cast<float4*>(p.S + slot * size + e + 4) = *reinterpret_cast<const float4*>(S + 4);
    }
    if (KIND == KIND_MLSTM && blockIdx.x == 0) {
        // normaliser and running maximum; m itself is stored by the output kernel (other blocks of this grid still read it)
        for (int c = threadIdx.x; c < dk; c += 256) {
            float nn = p.n[slot * dk + c], m = m0;
            constexpr int U = 8;
            for (int i0 = lo; i0 < hi; i0 += U) {
                float x[U], bc[U], mc[U];
#pragma unroll
                for (int j = 0; j < U; ++j) {
                    const size_t at = (size_t)(min(i0 + j, hi - 1) - cp.c0) * p.h + h;
                    x[j] = cp.nloc[at * dk + c];
                    bc[j] = cp.scal[at * 4];
                    mc[j] = cp.scal[at * 4 + 1];
                }
#pragma unroll
                for (int j = 0; j < U; ++j) {
                    if (i0 + j >= hi) break;
                    const size_t at = (size_t)(i0 + j - cp.c0) * p.h + h;
                    const float top = fmaxf(m, mc[j]);
                    cp.nloc[at * dk + c] = nn;
                    nn = expf(m - top) * nn + expf(mc[j] - top) * x[j];
                    if (c == 0) cp.scal[at * 4 + 2] = m;
                    m = bc[j] + top;
                    if (c == 0) cp.scal[at * 4 + 3] = m;
                }
            }
            p.n[slot * dk + c] = nn;
        }
    }
}

// ---- 3: outputs --------------------------------------------------------------------------------------------------------------
constexpr int OUT_THREADS = 512;             // 16 warps: 4 row tiles of 16 tokens x 4 column quarters
constexpr int LDA = CT + 8;

size_t output_smem(int kind, int dk, int dv, int slab, int bufs) {
    const int dkp = (dk + 15) / 16 * 16;
    const size_t slabs = (size_t)bufs * 2 * slab * (dv + 8) * 2, scores = (size_t)2 * CT * LDA * 2;
    size_t b = (size_t)CT * (dkp + 8) * 2 * 2 + (size_t)CT * (dv + 8) * 2 + (slabs > scores ? slabs : scores);
    b += kind == KIND_GLA ? (size_t)CT * (dkp + 4) * 4 : kind == KIND_RETENTION ? (size_t)CT * (dkp + 8) * 2 * 2 : 0;
    return b + (size_t)CT * 12 * 4;
}

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
    const GatedScanParams& p = cp.s;
    const int ci = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int rt = warp & 3, quarter = warp >> 2;
    const int* ch = cp.chunks + (size_t)(cp.c0 + ci) * 4;
    const int seq = ch[0], t0 = ch[1], n = ch[2], last = ch[3], dk = p.dk, dv = p.dv;
    const int dkp = (dk + 15) / 16 * 16, ldk = dkp + 8, ldv = dv + 8, ldb = dkp + 4;
    bf16* qs = reinterpret_cast<bf16*>(smraw);           // [CT][ldk]
    bf16* ks = qs + CT * ldk;
    bf16* vs = ks + CT * ldk;                            // [CT][ldv]
    bf16* slabs = vs + CT * ldv;                         // state rows [slab][ldv], high and low terms, one or two slabs; then
    bf16* ah = slabs;                                    // [CT][LDA] scores, high and low terms
    bf16* al = ah + CT * LDA;
    const int slab = cp.slab, region = max(cp.slab_bufs * 2 * slab * ldv, 2 * CT * LDA);
    float* fs = reinterpret_cast<float*>(slabs + region);
    float* bs = fs;                                      // GLA: [CT][ldb]
    bf16* ql = reinterpret_cast<bf16*>(fs);              // retention: [CT][ldk] low terms of the turned queries and keys
    bf16* kl = ql + CT * ldk;
    float* rows = fs + (KIND == KIND_GLA ? CT * ldb : KIND == KIND_RETENTION ? CT * ldk : 0);
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
    load_rows(qs, ldk, (const bf16*)p.q + (size_t)t0 * p.ld + h * dk, p.ld, n, dk, dkp);
    if (KIND == KIND_GLA) {
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
    load_rows(ks, ldk, (const bf16*)p.k + (size_t)t0 * p.ld + h * dk, p.ld, n, dk, dkp);
    load_rows(vs, ldv, (const bf16*)p.v + (size_t)t0 * p.ld + h * dv, p.ld, n, dv, dv);
    cp_async_commit();
    // a token's row, as it was loaded -> turned by its position, high and low terms
    auto turn_rows = [&](bf16* hi, bf16* lo) {
        const int per = dkp / 2;
        for (int i = tid; i < CT * per; i += OUT_THREADS) {
            const int r = i / per, c = i % per * 2;
            uint32_t a = 0, b = 0;
            if (r < n && c < dk) {
                const float2 x = turned(p, t0 + r, c, bf162_to_f2(*reinterpret_cast<const uint32_t*>(hi + r * ldk + c)));
                split_bf162(x.x, x.y, a, b);
            }
            *reinterpret_cast<uint32_t*>(hi + r * ldk + c) = a;
            *reinterpret_cast<uint32_t*>(lo + r * ldk + c) = b;
        }
    };
    const float rate = KIND == KIND_RETENTION ? p.decay[p.h + h] : 0.f;
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
    if (KIND == KIND_RETENTION) {
        turn_rows(qs, ql);
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
            if (KIND != KIND_GLA) {
                ldsm_x4(a, qs + (rt * 16 + (lane & 15)) * ldk + k0 + kk + (lane >> 4) * 8);
                if (KIND == KIND_RETENTION) ldsm_x4(a2, ql + (rt * 16 + (lane & 15)) * ldk + k0 + kk + (lane >> 4) * 8);
            } else {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int r = (i & 1) ? r1 : r0, c = k0 + kk + c4 * 2 + (i >> 1) * 8;
                    const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(qs + r * ldk + c));
                    const float2 b = *reinterpret_cast<const float2*>(bs + r * ldb + c);
                    split_bf162(x.x * qscale * exp2_fast(b.x), x.y * qscale * exp2_fast(b.y), a[i], a2[i]);
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
                if (KIND != KIND_MLSTM) mma_bf16_16816(acc[i], a2, b0, b1);
            }
        }
        if (k0 + cp.slab_bufs * slab < dkp) {
            __syncthreads();
            load_slab(k0 + cp.slab_bufs * slab);
            cp_async_commit();
        }
    }
    float e0 = 1.f, e1 = 1.f;
    if (KIND != KIND_GLA) {
        e0 = (KIND == KIND_MLSTM ? __expf(m_in - gx[r0]) : exp2f((float)(r0 + 1) * rate)) * qscale;
        e1 = (KIND == KIND_MLSTM ? __expf(m_in - gx[r1]) : exp2f((float)(r1 + 1) * rate)) * qscale;
#pragma unroll
        for (int i = 0; i < NT; ++i) { acc[i][0] *= e0; acc[i][1] *= e0; acc[i][2] *= e1; acc[i][3] *= e1; }
    }
    cp_async_wait<0>();
    __syncthreads();                                     // (the scores take the place of the state slabs)
    if (KIND == KIND_RETENTION) {
        turn_rows(ks, kl);
        __syncthreads();
    }
    // ---- scores of (row tile rt, key tile J = quarter) ----
    {
        const int J = quarter, r0 = rt * 16 + g, r1 = r0 + 8;
        float sc[2][4] = {};
        if (KIND != KIND_GLA ? J <= rt : J < rt) {
            for (int kk = 0; kk < dkp; kk += 16) {
                uint32_t a[4], a2[4];
                if (KIND != KIND_GLA) {
                    ldsm_x4(a, qs + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
                    if (KIND == KIND_RETENTION) ldsm_x4(a2, ql + (rt * 16 + (lane & 15)) * ldk + kk + (lane >> 4) * 8);
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
                    if (KIND != KIND_GLA) {
                        uint32_t b0, b1;
                        ldsm_x2(b0, b1, ks + (s + (lane & 7)) * ldk + kk + ((lane >> 3) & 1) * 8);
                        mma_bf16_16816(sc[t], a, b0, b1);
                        if (KIND == KIND_RETENTION) {
                            mma_bf16_16816(sc[t], a2, b0, b1);
                            ldsm_x2(b0, b1, kl + (s + (lane & 7)) * ldk + kk + ((lane >> 3) & 1) * 8);
                            mma_bf16_16816(sc[t], a, b0, b1);
                        }
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
        if (KIND != KIND_GLA || J != rt) {
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int t = 0; t < 2; ++t) {
                float v[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int r = i < 2 ? r0 : r1, s = J * 16 + t * 8 + c4 * 2 + (i & 1);
                    float w = qscale;
                    if (KIND == KIND_MLSTM) w *= s < n ? __expf(ga[s] - gx[r]) : 0.f;
                    if (KIND == KIND_RETENTION) w *= exp2f((float)max(r - s, 0) * rate);
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
    if (KIND == KIND_GLA) {
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
                a *= qscale;
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
        const float2 w = KIND == KIND_RETENTION ? make_float2(p.out_scale, p.out_scale) : make_float2(nw[j], nw[j + 1]);
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = u ? r1 : r0;
            if (r >= n) continue;
            const float inv = u ? i1 : i0;
            const float2 gt = bf162_to_f2(*reinterpret_cast<const uint32_t*>((const bf16*)p.g + (size_t)(t0 + r) * p.ld + h * dv + j));
            const float x = 1.f / (1.f + __expf(-gt.x)), y = 1.f / (1.f + __expf(-gt.y));
            const float gx0 = KIND == KIND_MLSTM ? x : gt.x * x, gy0 = KIND == KIND_MLSTM ? y : gt.y * y;
            *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)(t0 + r) * p.ldo + h * dv + j) =
                f2_to_bf162(acc[i][u * 2] * inv * w.x * gx0, acc[i][u * 2 + 1] * inv * w.y * gy0);
        }
    }
}

size_t state_smem(int kind, int dk, int dv, int rank) {
    const int dkp = (dk + 15) / 16 * 16;
    return (size_t)CT * (dkp + 8) * 4 + (size_t)CT * (dv + 8) * 2 + (kind == KIND_GLA ? (size_t)CT * (dk + rank) * 4 + (size_t)dk * rank * 2 : (size_t)3 * CT * 4);
}

template <int KIND>
int run_chunks(const GatedChunkParams* args, int B, cudaStream_t s) {
    GatedChunkParams params = *args;
    const size_t s3 = plan_output(KIND, args->s.dk, args->s.dv, params.slab, params.slab_bufs);
    const GatedChunkParams* p = &params;
    const int dk = p->s.dk, dv = p->s.dv, h = p->s.h, nc = p->c1 - p->c0;
    const size_t s1 = state_smem(KIND, dk, dv, p->s.rank);
    auto k1 = chunk_state_kernel<KIND>;
    if (s1 > 48 * 1024) cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    sl_launch(k1, dim3(nc, h), 256, s1, s, *p);
    sl_launch(chunk_scan_kernel<KIND>, dim3((dk * dv + 2047) / 2048, h, B), 256, 0, s, *p);
    if (dv <= 128) {
        auto k3 = chunk_output_kernel<KIND, 4>;
        cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        sl_launch(k3, dim3(nc, h), OUT_THREADS, s3, s, *p);
    } else {
        auto k3 = chunk_output_kernel<KIND, 8>;
        cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
        sl_launch(k3, dim3(nc, h), OUT_THREADS, s3, s, *p);
    }
    return SL_LAUNCH_CHECK();
}

}  // namespace

// 1 when the chunked kernels take these sizes (head rows of whole 16-byte pieces, tiles that fit in shared memory).
SL_API int sl_gated_chunk_ok(int kind, int dk, int dv, int rank) {
    if (dk < 8 || dv < 8 || dk % 8 != 0 || dv % 8 != 0 || dv > 256) return 0;
    int slab, bufs;
    return state_smem(kind, dk, dv, rank) <= SMEM_MAX && plan_output(kind, dk, dv, slab, bufs) <= SMEM_MAX;
}

// One pass over the chunks [c0, c1) of B sequences (bf16 rows in and out).  Passes of one step run in order on one stream.
SL_API int sl_gated_chunks(const GatedChunkParams* p, int B, int kind, cudaStream_t s) {
    if (B == 0 || p->c1 <= p->c0) return 0;
    if (!sl_gated_chunk_ok(kind, p->s.dk, p->s.dv, p->s.rank) || p->s.ld % 8 != 0 || B > 65535 || p->s.h > 65535) return -1;
    if (p->s.ldo % 2 != 0 || (uintptr_t)p->s.out % 4 != 0) return -1;
    if (kind == KIND_RETENTION) return p->s.rot_dims <= p->s.dk && p->s.rot_dims % 2 == 0 ? run_chunks<KIND_RETENTION>(p, B, s) : -1;
    return kind == KIND_GLA ? run_chunks<KIND_GLA>(p, B, s) : kind == KIND_MLSTM ? run_chunks<KIND_MLSTM>(p, B, s) : -1;
}
