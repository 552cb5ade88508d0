// Tensor-core kernels of latent attention (bf16 cache rows [latent | rotated key part], sliding window, softmax sink).
//
//  * latent_gather_kernel: the cache rows that a step's portions can see, copied out of the pages in order.
//  * portion_attn_kernel: attention of portions of prompts over gathered rows, also used by grouped-query attention.  In latent
//    attention it is the expanded form: keys and values of the visible rows were materialised per head by two GEMMs, and a
//    shared rotated key part may be read beside the head's own.  FlashAttention-2 style over 128 queries x 1 head per CTA, tiles
//    of 64 keys come through a three-stage cp.async ring filled by a warp of its own.  A sliding window may keep the sequence's
//    first tokens visible: their tiles come before the window's.
//  * latent_decode_kernel: absorbed form, one query token per page-table row.  A CTA takes 16 heads x a range of keys: all
//    heads share the key rows, whose first `rank` values are the value rows as well, so a tile is read once for both products.
//    Key splits leave (o, log-sum-exp) partials for `sl_combine_vexpand` / `sl_mla_combine`; the sink belongs to split 0.
//
// Scores and softmax are fp32; the weights enter the second product as two bf16 terms (hi + lo), so they keep fp32-like accuracy.
#include "common.cuh"
#include "mma_sync.cuh"
#include "tcgen05.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

struct LatentGatherParams {
    void* out;                            // [total, row]
    const bf16* cache; int num_slots, row;
    const int* ranges;                    // [B][4]: page-table row, first position, rows, first output row
    const int* page_table; int pt_stride, page_size;
    int* guard;
};

// grid (ceil(longest / 8), B), block 256: a warp per row
__global__ void __launch_bounds__(256) latent_gather_kernel(LatentGatherParams p) {
    pdl_grid_sync();
    const int* rg = p.ranges + blockIdx.y * 4;
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= rg[2]) return;
    const int kp = rg[1] + i;
    const long long slot = (long long)p.page_table[(size_t)rg[0] * p.pt_stride + kp / p.page_size] * p.page_size + kp % p.page_size;
    if (!guard_ok(p.guard, 23, slot, p.num_slots)) return;
    const uint4* src = reinterpret_cast<const uint4*>(p.cache + (size_t)slot * p.row);
    uint4* dst = reinterpret_cast<uint4*>((bf16*)p.out + (size_t)(rg[3] + i) * p.row);
    for (int c = lane; c < p.row / 8; c += 32) dst[c] = src[c];
}

struct PortionAttnParams {
    const bf16* q; int ldq, q_head;       // (unrotated) query of head i at i * q_head
    const bf16* q_rot;                    // [T, heads, rot_dim] (rot_dim 0: none)
    const bf16* k; int ldk;               // keys [rows, ldk], key head of h0 + i at (i / kv_group) * dim
    const bf16* v; int ldv;               // values, likewise at (i / kv_group) * vdim
    const bf16* rows; int row, rank;      // gathered cache rows: rotated key part at `rank`
    const int* tiles;                     // [tiles][5]: first token, tokens, position of the first token, (key row - key position)
                                          // of the window's keys and of the kept first ones
    int heads, h0, dim, rot_dim, vdim, kv_group, window, keep_first;
    float scale;
    const float* sink;                    // [heads] or null
    bf16* out; int ldo;                   // [T, ldo]: head i at i * vdim
    int* err;                             // status word: set when a wait inside the kernel expired
    int stages;                           // set by the launcher: key tiles in shared memory
    const float2* turn; int ldt;          // values that turned with their position: (cos, sin) by which the adjacent pair m of token
                                          // t's output is turned back, at t * ldt + m (or null)
    float out_scale;                      // factor on the output
};

constexpr int BQ = 128, BK = 64, MAX_STAGES = 3;
constexpr int CONSUMERS = BQ / 16, PT = (CONSUMERS + 1) * 32;      // a warp per 16 queries, one warp that fetches

// 16 bytes global -> shared, or zeros
__device__ __forceinline__ void cp_async16_or_zero(void* dst, const void* src, bool valid) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
// arrive on `bar` when all copies this thread has issued so far have landed (the barrier counts one arrival per thread)
__device__ __forceinline__ void cp_async_arrive(uint64_t* bar) {
    asm volatile("cp.async.mbarrier.arrive.noinc.shared.b64 [%0];" ::"r"(tc::smem_u32(bar)) : "memory");
}

__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// grid (heads of the group, tiles).  NT: 8-wide value tiles (vdim <= 8 * NT).  The fetching warp runs ahead of the consumers by
// up to `stages` key tiles; consumer warps do not wait for one another.
template <int NT>
__global__ void __launch_bounds__(PT, 1) portion_attn_kernel(PortionAttnParams p) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int hg = blockIdx.x, h = p.h0 + hg, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int* tl = p.tiles + (gridDim.y - 1 - blockIdx.y) * 5;      // late positions see most keys: start them first
    const int q0 = tl[0], nq = tl[1], pos0 = tl[2], koff = tl[3], koff_kept = tl[4], hk = hg / p.kv_group;
    const int dq = p.dim + p.rot_dim, dqp = (dq + 15) / 16 * 16, ld = dqp + 8, ldv = NT * 8 + 8;
    bf16* qs = reinterpret_cast<bf16*>(smraw);            // [BQ][ld]
    const int stages = p.stages;
    bf16* ks = qs + BQ * ld;                              // stages x [BK][ld]
    bf16* vs = ks + stages * BK * ld;                     // stages x [BK][ldv]
    __shared__ uint64_t full[MAX_STAGES], empty[MAX_STAGES];
    __shared__ int gave_up;
    const int nd = p.dim / 8, nr = p.rot_dim / 8, nv = p.vdim / 8;
    const int last = pos0 + nq - 1;
    const int first = p.window > 0 ? max(0, pos0 - p.window + 1) : 0;
    const int kept = min(p.keep_first, first), kept_tiles = (kept + BK - 1) / BK;      // kept keys in front of the tile's window
    const int ntiles = kept_tiles + (last - first) / BK + 1;
    auto tile_start = [&](int j) { return j < kept_tiles ? j * BK : first + (j - kept_tiles) * BK; };

    // columns that no copy writes: the query / key padding to 16 and the value padding
    for (int i = tid; i < (BQ + stages * BK) * (dqp - dq); i += PT) qs[(i / (dqp - dq)) * ld + dq + i % (dqp - dq)] = __float2bfloat16(0.f);
    const int vpad = NT * 8 - p.vdim;
    for (int i = tid; i < stages * BK * vpad; i += PT) vs[(i / vpad) * ldv + p.vdim + i % vpad] = __float2bfloat16(0.f);
    for (int i = tid; i < BQ * (nd + nr); i += PT) {
        const int r = i / (nd + nr), c = i % (nd + nr);
        uint4 x = make_uint4(0, 0, 0, 0);
        if (r < nq)
            x = c < nd ? *reinterpret_cast<const uint4*>(p.q + (size_t)(q0 + r) * p.ldq + (size_t)h * p.q_head + c * 8)
                       : *reinterpret_cast<const uint4*>(p.q_rot + ((size_t)(q0 + r) * p.heads + h) * p.rot_dim + (c - nd) * 8);
        *reinterpret_cast<uint4*>(qs + r * ld + c * 8) = x;
    }
    if (tid == 0) {
        gave_up = 0;
        for (int i = 0; i < stages; ++i) {
            tc::mbar_init(&full[i], 32);
            tc::mbar_init(&empty[i], CONSUMERS);
        }
        tc::mbar_fence_init();
    }
    __syncthreads();
    volatile int* dead = &gave_up;                        // a wait expired somewhere in the block: nobody waits any longer
    auto wait = [&](uint64_t* bar, int parity) {
        if (tc::mbar_wait(bar, parity) || *dead) return;
        *dead = 1;
        if (p.err != nullptr) atomicCAS(p.err, 0, 41);
    };
    if (warp == CONSUMERS) {
        // a lane copies the same 16-byte column of every (32 / pieces)-th row of a part (a row has at most 32 pieces)
        struct Part { int row, step; bool on; };
        auto part = [&](int pieces) {
            Part x;
            x.step = pieces > 0 ? 32 / pieces : 1;
            x.row = pieces > 0 ? lane / pieces : 0;
            x.on = pieces > 0 && x.row < x.step;
            return x;
        };
        const Part pk = part(nd), pr = part(nr), pv = part(nv);
        const bf16* kcol = p.k + hk * p.dim + lane % nd * 8;
        const bf16* rcol = nr > 0 ? p.rows + p.rank + lane % nr * 8 : nullptr;
        const bf16* vcol = p.v + hk * p.vdim + lane % nv * 8;
        auto copy = [&](const Part& x, bf16* dst, int dld, const bf16* col, size_t sld, int k0, int n, int off) {
            if (!x.on) return;
            const bf16* src = col + (ptrdiff_t)(k0 + x.row + off) * (ptrdiff_t)sld;
            dst += x.row * dld;
            const int dstep = x.step * dld;
            const size_t sstep = (size_t)x.step * sld;
            int r = x.row;
#pragma unroll 4
            for (; r < n; r += x.step, src += sstep, dst += dstep) cp_async16(dst, src);
            for (; r < BK; r += x.step, dst += dstep) cp_async16_or_zero(dst, col, false);
        };
        for (int j = 0; j < ntiles && !*dead; ++j) {
            const int st = j % stages, k0 = tile_start(j), n = min(BK, (j < kept_tiles ? kept : last + 1) - k0);
            const int off = j < kept_tiles ? koff_kept : koff;
            if (j >= stages) wait(&empty[st], (j / stages - 1) & 1);
            bf16* kd = ks + st * BK * ld;
            bf16* vd = vs + st * BK * ldv;
            copy(pk, kd + lane % nd * 8, ld, kcol, p.ldk, k0, n, off);
            if (nr > 0) copy(pr, kd + p.dim + lane % nr * 8, ld, rcol, p.row, k0, n, off);
            copy(pv, vd + lane % nv * 8, ldv, vcol, p.ldv, k0, n, off);
            cp_async_arrive(&full[st]);
        }
        cp_async_wait_all();
        return;
    }

    const int r0 = warp * 16 + g, r1 = r0 + 8, p0 = pos0 + r0, p1 = pos0 + r1;
    const int lo0 = p.window > 0 ? p0 - p.window + 1 : 0, lo1 = p.window > 0 ? p1 - p.window + 1 : 0;
    const float scale_log2 = p.scale * LOG2E;
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
    if (p.sink != nullptr) { m0 = m1 = p.sink[h] * LOG2E; l0 = l1 = 1.f; }
    const int wq0 = pos0 + warp * 16, wlo = p.window > 0 ? wq0 - p.window + 1 : 0;      // range of the warp's rows

    for (int j = 0; j < ntiles; ++j) {
        const int st = j % stages;
        wait(&full[st], (j / stages) & 1);
        if (*dead) break;
        const bf16* kt = ks + st * BK * ld;
        const bf16* vt = vs + st * BK * ldv;
        const int k0 = tile_start(j), ke = j < kept_tiles ? kept : last + 1;
        if (warp * 16 < nq && (j < kept_tiles || (k0 <= wq0 + 15 && (k0 + BK - 1 >= wlo || k0 < p.keep_first)))) {      // it meets the warp's rows
            float s[BK / 8][4];
#pragma unroll
            for (int n = 0; n < BK / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            for (int kk = 0; kk < dqp; kk += 16) {
                uint32_t a[4];
                ldsm_x4(a, qs + (warp * 16 + (lane & 15)) * ld + kk + (lane >> 4) * 8);
#pragma unroll
                for (int n = 0; n < BK / 16; ++n) {
                    uint32_t b[4];                         // two key tiles: lanes 0-15 address the first, 16-31 the second
                    ldsm_x4(b, kt + (n * 16 + (lane & 7) + (lane >> 4) * 8) * ld + kk + ((lane >> 3) & 1) * 8);
                    mma_bf16_16816(s[2 * n], a, b[0], b[1]);
                    mma_bf16_16816(s[2 * n + 1], a, b[2], b[3]);
                }
            }
            const int kl = k0 + BK - 1;                    // every row of the warp sees every key of the tile
            const bool whole = kl < ke && kl <= wq0 && (k0 >= wlo + 15 || kl < p.keep_first);
            float x0 = m0, x1 = m1;
            if (whole) {
#pragma unroll
                for (int n = 0; n < BK / 8; ++n) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) s[n][i] *= scale_log2;
                }
            } else {
                const int hi0 = min(p0, ke - 1), hi1 = min(p1, ke - 1);
#pragma unroll
                for (int n = 0; n < BK / 8; ++n) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int key = k0 + n * 8 + 2 * c4 + (i & 1);
                        const bool in = i < 2 ? (key <= hi0 && (key >= lo0 || key < p.keep_first))
                                              : (key <= hi1 && (key >= lo1 || key < p.keep_first));
                        s[n][i] = in ? s[n][i] * scale_log2 : -INFINITY;
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < BK / 8; ++n) {
                x0 = fmaxf(x0, fmaxf(s[n][0], s[n][1]));
                x1 = fmaxf(x1, fmaxf(s[n][2], s[n][3]));
            }
            x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1)); x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
            x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1)); x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
            const float f0 = m0 == -INFINITY ? 0.f : exp2f(m0 - x0), f1 = m1 == -INFINITY ? 0.f : exp2f(m1 - x1);
            const float z0 = x0 == -INFINITY ? 0.f : x0, z1 = x1 == -INFINITY ? 0.f : x1;      // (a row may see no key of this tile)
            m0 = x0; m1 = x1;
            float sum0 = 0.f, sum1 = 0.f;
#pragma unroll
            for (int i = 0; i < NT; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
#pragma unroll
            for (int n = 0; n < BK / 16; ++n) {
                uint32_t ph[4], pl[4];
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    float* sn = s[2 * n + u];
                    const float e0 = exp2_fast(sn[0] - z0), e1 = exp2_fast(sn[1] - z0), e2 = exp2_fast(sn[2] - z1), e3 = exp2_fast(sn[3] - z1);
                    sum0 += e0 + e1;
                    sum1 += e2 + e3;
                    split_bf162(e0, e1, ph[u * 2], pl[u * 2]);
                    split_bf162(e2, e3, ph[u * 2 + 1], pl[u * 2 + 1]);
                }
#pragma unroll
                for (int i = 0; i < NT; i += 2) {
                    uint32_t b[4];                         // two value tiles
                    ldsm_x4_trans(b, vt + (n * 16 + (lane & 15)) * ldv + i * 8 + (lane >> 4) * 8);
                    mma_bf16_16816(acc[i], ph, b[0], b[1]);
                    mma_bf16_16816(acc[i], pl, b[0], b[1]);
                    mma_bf16_16816(acc[i + 1], ph, b[2], b[3]);
                    mma_bf16_16816(acc[i + 1], pl, b[2], b[3]);
                }
            }
            sum0 += __shfl_xor_sync(0xffffffffu, sum0, 1); sum0 += __shfl_xor_sync(0xffffffffu, sum0, 2);
            sum1 += __shfl_xor_sync(0xffffffffu, sum1, 1); sum1 += __shfl_xor_sync(0xffffffffu, sum1, 2);
            l0 = l0 * f0 + sum0;
            l1 = l1 * f1 + sum1;
        }
        __syncwarp();
        if (lane == 0) tc::mbar_arrive(&empty[st]);
    }
    const float i0 = l0 > 0.f ? p.out_scale / l0 : 0.f, i1 = l1 > 0.f ? p.out_scale / l1 : 0.f;
    auto store = [&](int r, int d, float x, float y) {
        if (r >= nq) return;
        if (p.turn != nullptr) {
            const float2 cs = p.turn[(size_t)(q0 + r) * p.ldt + (d >> 1)];
            const float a = x * cs.x + y * cs.y;
            y = y * cs.x - x * cs.y;
            x = a;
        }
        *reinterpret_cast<uint32_t*>(p.out + (size_t)(q0 + r) * p.ldo + (size_t)h * p.vdim + d) = f2_to_bf162(x, y);
    };
#pragma unroll
    for (int i = 0; i < NT; ++i) {
        const int d = i * 8 + 2 * c4;
        if (d >= p.vdim) break;
        store(r0, d, acc[i][0] * i0, acc[i][1] * i0);
        store(r1, d, acc[i][2] * i1, acc[i][3] * i1);
    }
}

int value_tiles(int vdim) { return vdim <= 32 ? 4 : vdim <= 64 ? 8 : vdim <= 128 ? 16 : 32; }
size_t prefill_smem(int dq, int nt, int stages) {
    const int ld = (dq + 15) / 16 * 16 + 8;
    return ((size_t)(BQ + stages * BK) * ld + (size_t)stages * BK * (nt * 8 + 8)) * sizeof(bf16);
}
constexpr size_t SMEM_MAX = 224 * 1024;
int prefill_stages(int dq, int nt) { return prefill_smem(dq, nt, MAX_STAGES) <= SMEM_MAX ? MAX_STAGES : 2; }

constexpr int DK_T = 64;                  // keys per tile of the decode kernel

struct LatentDecodeParams {
    const bf16* q_abs;                    // [T, heads, rank]
    const bf16* q_rot;                    // [T, heads, rot_dim]
    const bf16* cache; int num_slots;
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    int heads, rank, rot_dim, window, splits;
    float scale;
    const float* sink;
    float* o_part; float* lse_part;       // [T, heads, splits, rank], [T, heads, splits]
    bf16* o_final;                        // [T, heads, rank] instead, with one split
    int* guard;
};

// grid (splits, head groups of 16, T), block 256.  NTW: 8-wide value tiles per warp (rank <= 64 * NTW).
template <int NTW>
__global__ void __launch_bounds__(256) latent_decode_kernel(LatentDecodeParams p) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int split = blockIdx.x, h0 = blockIdx.y * 16, t = blockIdx.z;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int row = p.rank + p.rot_dim, dqp = (row + 15) / 16 * 16, ld = dqp + 8;
    bf16* qs = reinterpret_cast<bf16*>(smraw);            // [16][ld]
    bf16* ks = qs + 16 * ld;                              // [DK_T][ld]
    float* sc = reinterpret_cast<float*>(ks + DK_T * ld);   // [16][DK_T + 4]
    bf16* ph = reinterpret_cast<bf16*>(sc + 16 * (DK_T + 4));      // [16][DK_T + 8]
    bf16* pl = ph + 16 * (DK_T + 8);
    float* fac = reinterpret_cast<float*>(pl + 16 * (DK_T + 8));   // [16] rescale of the tile, then 1 / l
    const int pos = p.positions[t];
    const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    const int tiles = (pos - first) / DK_T + 1, per = (tiles + p.splits - 1) / p.splits;
    const int tb = min(tiles, split * per), te = min(tiles, tb + per);
    const int* pt = p.page_table + (size_t)p.batch_idx[t] * p.pt_stride;
    for (int i = tid; i < 16 * (dqp / 8); i += 256) {
        const int r = i / (dqp / 8), c = (i % (dqp / 8)) * 8;
        uint4 x = make_uint4(0, 0, 0, 0);
        if (h0 + r < p.heads && c < row)
            x = c < p.rank ? *reinterpret_cast<const uint4*>(p.q_abs + ((size_t)t * p.heads + h0 + r) * p.rank + c)
                           : *reinterpret_cast<const uint4*>(p.q_rot + ((size_t)t * p.heads + h0 + r) * p.rot_dim + c - p.rank);
        *reinterpret_cast<uint4*>(qs + r * ld + c) = x;
    }
    if (dqp > row && tid < DK_T) *reinterpret_cast<uint4*>(ks + tid * ld + row) = make_uint4(0, 0, 0, 0);     // (row % 8 == 0)
    float m[2], l[2];                                     // softmax state of rows 2 * warp, 2 * warp + 1
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int h = h0 + warp * 2 + u;
        const bool s = split == 0 && p.sink != nullptr && h < p.heads;
        m[u] = s ? p.sink[h] * LOG2E : -INFINITY;
        l[u] = s ? 1.f : 0.f;
    }
    const int nt = p.rank / 8, tw = (nt + 7) / 8, n0 = warp * tw, nn = max(0, min(tw, nt - n0));
    float acc[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const float scale_log2 = p.scale * LOG2E;
    for (int j = tb; j < te; ++j) {
        const int k0 = first + j * DK_T, nk = min(DK_T, pos + 1 - k0);
        __syncthreads();
        long long slot = -1;                              // lanes 0-7: the warp's eight rows
        if (lane < 8 && warp * 8 + lane < nk) {
            const int kp = k0 + warp * 8 + lane;
            const long long s = (long long)pt[kp / p.page_size] * p.page_size + kp % p.page_size;
            slot = guard_ok(p.guard, 24, s, p.num_slots) ? s : -1;
        }
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            const long long s = __shfl_sync(0xffffffffu, slot, r);
            bf16* dst = ks + (warp * 8 + r) * ld;
            const bf16* src = p.cache + (size_t)(s < 0 ? 0 : s) * row;
            for (int c = lane * 8; c < row; c += 256) {
                if (s >= 0) cp_async16(dst + c, src + c);
                else *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
            }
        }
        cp_async_commit();
        cp_async_wait<0>();
        __syncthreads();
        float s4[4] = {0.f, 0.f, 0.f, 0.f};               // 16 heads x the warp's eight keys
        for (int kk = 0; kk < dqp; kk += 16) {
            uint32_t a[4], b0, b1;
            ldsm_x4(a, qs + (lane & 15) * ld + kk + (lane >> 4) * 8);
            ldsm_x2(b0, b1, ks + (warp * 8 + (lane & 7)) * ld + kk + ((lane >> 3) & 1) * 8);
            mma_bf16_16816(s4, a, b0, b1);
        }
        {
            const int kc = warp * 8 + c4 * 2;
            sc[g * (DK_T + 4) + kc] = kc < nk ? s4[0] * scale_log2 : -INFINITY;
            sc[g * (DK_T + 4) + kc + 1] = kc + 1 < nk ? s4[1] * scale_log2 : -INFINITY;
            sc[(g + 8) * (DK_T + 4) + kc] = kc < nk ? s4[2] * scale_log2 : -INFINITY;
            sc[(g + 8) * (DK_T + 4) + kc + 1] = kc + 1 < nk ? s4[3] * scale_log2 : -INFINITY;
        }
        __syncthreads();
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int r = warp * 2 + u;
            const float2 v = *reinterpret_cast<const float2*>(sc + r * (DK_T + 4) + lane * 2);
            const float x = fmaxf(m[u], warp_max(fmaxf(v.x, v.y)));
            const float f = m[u] == -INFINITY ? 0.f : exp2f(m[u] - x);
            const float e0 = exp2f(v.x - x), e1 = exp2f(v.y - x);
            l[u] = l[u] * f + warp_sum(e0 + e1);
            m[u] = x;
            uint32_t hi, lo;
            split_bf162(e0, e1, hi, lo);
            *reinterpret_cast<uint32_t*>(ph + r * (DK_T + 8) + lane * 2) = hi;
            *reinterpret_cast<uint32_t*>(pl + r * (DK_T + 8) + lane * 2) = lo;
            if (lane == 0) fac[r] = f;
        }
        __syncthreads();
        const float f0 = fac[g], f1 = fac[g + 8];
#pragma unroll
        for (int i = 0; i < NTW; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
#pragma unroll
        for (int kk = 0; kk < DK_T; kk += 16) {
            uint32_t a[4], a2[4];
            ldsm_x4(a, ph + (lane & 15) * (DK_T + 8) + kk + (lane >> 4) * 8);
            ldsm_x4(a2, pl + (lane & 15) * (DK_T + 8) + kk + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                if (i >= nn) break;
                uint32_t b0, b1;
                ldsm_x2_trans(b0, b1, ks + (kk + (lane & 15)) * ld + (n0 + i) * 8);
                mma_bf16_16816(acc[i], a, b0, b1);
                mma_bf16_16816(acc[i], a2, b0, b1);
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < 2; ++u) {
        const int r = warp * 2 + u, h = h0 + r;
        if (lane == 0) {
            fac[r] = l[u] > 0.f ? 1.f / l[u] : 0.f;
            if (h < p.heads && p.lse_part != nullptr)
                p.lse_part[((size_t)t * p.heads + h) * p.splits + split] = l[u] > 0.f ? (m[u] + log2f(l[u])) / LOG2E : -INFINITY;
        }
    }
    __syncthreads();
    const float i0 = fac[g], i1 = fac[g + 8];
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
        if (i >= nn) break;
        const int d = (n0 + i) * 8 + c4 * 2;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int h = h0 + g + u * 8;
            if (h >= p.heads) continue;
            const float inv = u ? i1 : i0, x = acc[i][u * 2] * inv, y = acc[i][u * 2 + 1] * inv;
            if (p.o_final != nullptr) *reinterpret_cast<uint32_t*>(p.o_final + ((size_t)t * p.heads + h) * p.rank + d) = f2_to_bf162(x, y);
            else *reinterpret_cast<float2*>(p.o_part + (((size_t)t * p.heads + h) * p.splits + split) * p.rank + d) = make_float2(x, y);
        }
    }
}

size_t decode_smem(int row) {
    const int ld = (row + 15) / 16 * 16 + 8;
    return (size_t)(16 + DK_T) * ld * 2 + (size_t)16 * (DK_T + 4) * 4 + (size_t)2 * 16 * (DK_T + 8) * 2 + 64;
}

}  // namespace

SL_API int sl_latent_gather(const LatentGatherParams* p, int B, int longest, cudaStream_t s) {
    if (B == 0 || longest == 0) return 0;
    if (p->row % 8 != 0 || B > 65535) return -1;
    sl_launch(latent_gather_kernel, dim3((longest + 7) / 8, B), 256, 0, s, *p);
    return SL_LAUNCH_CHECK();
}

// 1 when portion_attn_kernel takes these sizes.
SL_API int sl_portion_attn_ok(int dim, int rot_dim, int vdim) {
    if (dim < 8 || rot_dim < 0 || vdim < 8 || dim % 8 != 0 || rot_dim % 8 != 0 || vdim % 8 != 0 || vdim > 256 || dim + rot_dim > 256) return 0;
    return prefill_smem(dim + rot_dim, value_tiles(vdim), 2) <= SMEM_MAX;
}

// 1 when the tensor-core kernels of latent attention take these sizes.
SL_API int sl_latent_mma_ok(int dim, int rot_dim, int vdim, int rank) {
    return sl_portion_attn_ok(dim, rot_dim, vdim) && rank >= 8 && rank % 8 == 0 && rank <= 1024 && decode_smem(rank + rot_dim) <= SMEM_MAX;
}

// `heads` of the launch are h0 .. h0 + group - 1.
SL_API int sl_portion_attn(const PortionAttnParams* args, int group, int tiles, cudaStream_t s) {
    PortionAttnParams params = *args;
    PortionAttnParams* p = &params;
    if (group == 0 || tiles == 0) return 0;
    if (!sl_portion_attn_ok(p->dim, p->rot_dim, p->vdim) || tiles > 65535 || p->kv_group < 1) return -1;
    if (((uintptr_t)p->k | (uintptr_t)p->v | (uintptr_t)p->q) % 16 != 0 || ((uintptr_t)p->out | (uintptr_t)(p->ldo * 2)) % 4 != 0) return -1;
    if (p->rot_dim > 0 && (((uintptr_t)p->rows | (uintptr_t)p->q_rot) % 16 != 0 || p->row % 8 != 0 || p->rank % 8 != 0)) return -1;
    if (p->ldq % 8 != 0 || p->q_head % 8 != 0 || p->ldk % 8 != 0 || p->ldv % 8 != 0) return -1;
    const int nt = value_tiles(p->vdim), dq = p->dim + p->rot_dim;
    p->stages = prefill_stages(dq, nt);
    const size_t smem = prefill_smem(dq, nt, p->stages);
#define SL_LP(NT)                                                                                                       \
    {                                                                                                                   \
        auto kern = portion_attn_kernel<NT>;                                                                          \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                             \
        sl_launch(kern, dim3(group, tiles), PT, smem, s, *p);                                                          \
    }
    if (nt == 4) SL_LP(4) else if (nt == 8) SL_LP(8) else if (nt == 16) SL_LP(16) else SL_LP(32)
#undef SL_LP
    return SL_LAUNCH_CHECK();
}

SL_API int sl_latent_decode(const LatentDecodeParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->rank % 8 != 0 || p->rot_dim % 8 != 0 || p->rank > 1024 || p->splits < 1 || T > 65535) return -1;
    if (p->o_final != nullptr && p->splits != 1) return -1;
    const size_t smem = decode_smem(p->rank + p->rot_dim);
    if (smem > SMEM_MAX) return -1;
    const dim3 grid(p->splits, (p->heads + 15) / 16, T);
#define SL_LD(NTW)                                                                                                      \
    {                                                                                                                   \
        auto kern = latent_decode_kernel<NTW>;                                                                          \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                             \
        sl_launch(kern, grid, 256, smem, s, *p);                                                                        \
    }
    if (p->rank <= 128) SL_LD(2) else if (p->rank <= 256) SL_LD(4) else if (p->rank <= 512) SL_LD(8) else SL_LD(16)
#undef SL_LD
    return SL_LAUNCH_CHECK();
}
