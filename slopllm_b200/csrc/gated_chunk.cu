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
// in three launches:
//   1 chunk_state_kernel   (chunk, head): decays, the chunk's own state contribution
//   2 chunk_scan_kernel    (elements, head, sequence): carries the fp32 state over the chunks and leaves each chunk's S_in
//   3 chunk_output_kernel  (chunk, head): intra-chunk and S_in parts, normaliser, head norm, output gate
//
// No exponent is ever positive: the products e^{b_t - b_s} of GLA are taken directly inside 16-token diagonal blocks and
// through an anchor between the blocks otherwise.  q, k, v come as bf16; every other operand of a tensor-core product (decayed
// keys and queries, scores, the state) is split into two bf16 terms, so the results keep fp32-like accuracy.
#include "gated_chunk.cuh"

namespace {

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
    } else if (warp == 0) {
        mlstm_gates(p, t0, n, h, fs, fs + CT, fs + 2 * CT);
    }
    cp_async_wait<0>();
    __syncthreads();
    const float top = KIND == KIND_MLSTM ? fs[2 * CT + n - 1] : 0.f;
    for (int i = tid; i < CT * (dkp / 2); i += 256) {
        const int s = i / (dkp / 2), c = (i % (dkp / 2)) * 2;
        uint32_t hi = 0, lo = 0;
        if (s < n && c < dk) {
            const float2 k = bf162_to_f2(*reinterpret_cast<const uint32_t*>(kh + s * ldk + c));
            float w0, w1;
            if (KIND == KIND_GLA) {
                w0 = exp2_fast(fs[(n - 1) * dk + c] - fs[s * dk + c]);
                w1 = exp2_fast(fs[(n - 1) * dk + c + 1] - fs[s * dk + c + 1]);
            } else {
                w0 = w1 = __expf(fs[s] - top);
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
                    d[j] = cp.b[(size_t)(ch[1] + ch[2] - 1) * (p.h * dk) + h * dk + c];
                }
            }
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const int i = i0 + j;
                if (i >= hi) break;
                float add = 1.f, keep = KIND == KIND_GLA ? exp2f(d[j]) : 1.f;
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
    return kind == KIND_GLA ? run_chunks<KIND_GLA>(p, B, s) : kind == KIND_MLSTM ? run_chunks<KIND_MLSTM>(p, B, s) : -1;
}
