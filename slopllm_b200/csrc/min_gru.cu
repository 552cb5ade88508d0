// minGRU: an element-wise gated recurrence whose gates read the current token only (sm_100a):
//
//   z = sigmoid(z_raw + b_z),  u = u_raw + b_u,  c = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S_t = (1 - z_t) S_{t-1} + z_t c_t,   out_t = S_t * silu(g_t)
//
// Gates, candidates, states and their products are fp32; rows and `out` are bf16 or fp32.
//
//  * min_gru_step_kernel: a thread walks a sequence's tokens for VW channels: decoding and short portions, one launch.
//  * min_gru_chunk_kernel, min_gru_apply_kernel: longer portions in chunks of 64 tokens.  A chunk maps the state that enters it to
//    A S + B; the first kernel makes (A, B) of every chunk, the second composes those in front of its own chunk and walks it.
//    Inside a chunk the warps' eight tokens are composed the same way, so no thread waits for more than eight tokens.
#include "common.cuh"

namespace {

struct MinGruParams {
    void* out; int ldo;                      // [T, W]
    const void *z, *u, *g; int ld;           // token-major rows
    const float *z_b, *u_b;                  // [W] or null
    float* S;                                // [slots, W]
    const int* qo_indptr; const int* state_idx;
    int W;
    const int* chunks; const int* seq_chunks;      // [chunks][4]: sequence, first token, tokens, 1 if the sequence's last; [B + 1]
    float2* maps;                            // [chunks, W]: (A, B) of each chunk
    float* start;                            // [B, W]: the state in front of each sequence's portion
};

template <int VW>
struct Row { float v[VW]; };
template <int VW>
__device__ __forceinline__ Row<VW> ld(const float* p) {
    Row<VW> r;
    if (VW == 4) {
        const float4 x = *reinterpret_cast<const float4*>(p);
        r.v[0] = x.x; r.v[VW / 4] = x.y; r.v[VW / 2] = x.z; r.v[VW - 1] = x.w;
    } else if (VW == 2) {
        const float2 x = *reinterpret_cast<const float2*>(p);
        r.v[0] = x.x; r.v[VW - 1] = x.y;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <int VW>
__device__ __forceinline__ Row<VW> ld(const bf16* p) {
    Row<VW> r;
    if (VW == 4) {
        const uint2 x = *reinterpret_cast<const uint2*>(p);
        const float2 a = bf162_to_f2(x.x), b = bf162_to_f2(x.y);
        r.v[0] = a.x; r.v[VW / 4] = a.y; r.v[VW / 2] = b.x; r.v[VW - 1] = b.y;
    } else if (VW == 2) {
        const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(p));
        r.v[0] = x.x; r.v[VW - 1] = x.y;
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int VW>
__device__ __forceinline__ void st(float* p, const Row<VW>& r) {
    if (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[VW / 4], r.v[VW / 2], r.v[VW - 1]);
    else if (VW == 2) *reinterpret_cast<float2*>(p) = make_float2(r.v[0], r.v[VW - 1]);
    else *p = r.v[0];
}
template <int VW>
__device__ __forceinline__ void st(bf16* p, const Row<VW>& r) {
    if (VW == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162(r.v[0], r.v[VW / 4]), f2_to_bf162(r.v[VW / 2], r.v[VW - 1]));
    else if (VW == 2) *reinterpret_cast<uint32_t*>(p) = f2_to_bf162(r.v[0], r.v[VW - 1]);
    else *p = __float2bfloat16(r.v[0]);
}

__device__ __forceinline__ float sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
// S <- a S + b of one token and channel
__device__ __forceinline__ float2 gate(float z_raw, float u) {
    const float z = sigmoid(z_raw), c = u >= 0.f ? u + 0.5f : sigmoid(u);
    return make_float2(1.f - z, z * c);
}

// The same for bf16 rows: hardware exponential and reciprocal (a few ulp), which do most of the work of a long portion.
constexpr float LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float exp2_fast(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float rcp_fast(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float silu_fast(float x) { return x * rcp_fast(1.f + exp2_fast(x * -LOG2E)); }
// zn: -log2(e) (z_raw).  Both sigmoids share one reciprocal; the bound on u's exponential keeps their product finite wherever z counts.
__device__ __forceinline__ float2 gate_fast(float zn, float u) {
    const float a = 1.f + exp2_fast(zn), b = 1.f + exp2_fast(fminf(u * -LOG2E, 62.f)), r = rcp_fast(a * b), z = r * b;
    return make_float2(1.f - z, u >= 0.f ? z * (u + 0.5f) : r);
}

// grid (ceil(W / (128 * VW)), B), block 128
template <int VW, typename TI, typename TO>
__global__ void __launch_bounds__(128) min_gru_step_kernel(MinGruParams p) {
    pdl_grid_sync();
    const int c = (blockIdx.x * 128 + threadIdx.x) * VW, seq = blockIdx.y;
    const int t0 = p.qo_indptr[seq], t1 = p.qo_indptr[seq + 1];
    if (c >= p.W || t0 >= t1) return;
    float* Sp = p.S + (size_t)p.state_idx[seq] * p.W + c;
    Row<VW> S = ld<VW>(Sp), zb{}, ub{};
    if (p.z_b != nullptr) zb = ld<VW>(p.z_b + c);
    if (p.u_b != nullptr) ub = ld<VW>(p.u_b + c);
    for (int t = t0; t < t1; ++t) {
        const size_t at = (size_t)t * p.ld + c;
        const Row<VW> z = ld<VW>((const TI*)p.z + at), u = ld<VW>((const TI*)p.u + at), g = ld<VW>((const TI*)p.g + at);
        Row<VW> o;
#pragma unroll
        for (int i = 0; i < VW; ++i) {
            const float2 m = gate(z.v[i] + zb.v[i], u.v[i] + ub.v[i]);
            S.v[i] = m.x * S.v[i] + m.y;
            o.v[i] = S.v[i] * g.v[i] * sigmoid(g.v[i]);
        }
        st<VW>((TO*)p.out + (size_t)t * p.ldo + c, o);
    }
    st<VW>(Sp, S);
}

// ---- chunks: a block takes 32 * VW channels of one chunk, a warp eight consecutive tokens of it ----
constexpr int CT = 64, WT = 8, WARPS = CT / WT;      // tokens of a chunk, tokens per warp

// (A, B) of the composition "first, then second"
__device__ __forceinline__ float2 then(float2 first, float2 second) { return make_float2(second.x * first.x, second.x * first.y + second.y); }

// The row of a warp's token t out of n; tokens behind the last read that one again, so that no load depends on a branch.
__device__ __forceinline__ int row_of(int t, int n) { return max(0, min(t, n - 1)); }

// All gates of a warp's tokens: every load is issued before the first is used.  `all`: their composition.
template <int VW, typename TI>
struct WarpGates {
    float2 m[WT][VW];
    float2 all[VW];
    __device__ __forceinline__ void load(const MinGruParams& p, int c, int t0, int n, const Row<VW>& zb, const Row<VW>& ub) {
        const TI *z = (const TI*)p.z + (size_t)t0 * p.ld + c, *u = (const TI*)p.u + (size_t)t0 * p.ld + c;
        Row<VW> zr[WT], ur[WT];
#pragma unroll
        for (int t = 0; t < WT; ++t) {
            zr[t] = ld<VW>(z + (size_t)row_of(t, n) * p.ld);
            ur[t] = ld<VW>(u + (size_t)row_of(t, n) * p.ld);
        }
#pragma unroll
        for (int i = 0; i < VW; ++i) all[i] = make_float2(1.f, 0.f);
#pragma unroll
        for (int t = 0; t < WT; ++t)
#pragma unroll
            for (int i = 0; i < VW; ++i) {
                const float u1 = ur[t].v[i] + ub.v[i];
                const float2 x = sizeof(TI) == 2 ? gate_fast(fmaf(zr[t].v[i], -LOG2E, zb.v[i] * -LOG2E), u1) : gate(zr[t].v[i] + zb.v[i], u1);
                m[t][i] = t < n ? x : make_float2(1.f, 0.f);
                all[i] = then(all[i], m[t][i]);
            }
    }
};

// grid (ceil(W / (32 * VW)), chunks), block 256
template <int VW, typename TI>
__global__ void __launch_bounds__(256) min_gru_chunk_kernel(MinGruParams p) {
    pdl_grid_sync();
    __shared__ float2 maps[WARPS][32 * VW];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x * 32 + lane) * VW;
    const int* ch = p.chunks + (size_t)blockIdx.y * 4;
    const int seq = ch[0], t0 = ch[1], n = ch[2];
    const bool in = c < p.W;
    if (in && warp == 0 && (int)blockIdx.y == p.seq_chunks[seq])     // (the second kernel overwrites the state while others need it)
        st<VW>(p.start + (size_t)seq * p.W + c, ld<VW>(p.S + (size_t)p.state_idx[seq] * p.W + c));
    if (ch[3]) return;                                               // nobody follows
    Row<VW> zb{}, ub{};
    WarpGates<VW, TI> g;
    if (in) {
        if (p.z_b != nullptr) zb = ld<VW>(p.z_b + c);
        if (p.u_b != nullptr) ub = ld<VW>(p.u_b + c);
        g.load(p, c, t0 + min(warp * WT, n - 1), n - warp * WT, zb, ub);
#pragma unroll
        for (int i = 0; i < VW; ++i) maps[warp][lane * VW + i] = g.all[i];
    }
    __syncthreads();
    if (!in || warp != 0) return;
    float2* out = p.maps + (size_t)blockIdx.y * p.W + c;
#pragma unroll
    for (int i = 0; i < VW; ++i) {
        float2 x = g.all[i];
#pragma unroll
        for (int w = 1; w < WARPS; ++w) x = then(x, maps[w][lane * VW + i]);
        out[i] = x;
    }
}

// the same grid; late chunks have most to compose: they start first
template <int VW, typename TI, typename TO>
__global__ void __launch_bounds__(256) min_gru_apply_kernel(MinGruParams p) {
    pdl_grid_sync();
    __shared__ float2 before[WARPS][32 * VW], maps[WARPS][32 * VW];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x * 32 + lane) * VW, ci = gridDim.y - 1 - blockIdx.y;
    const int* ch = p.chunks + (size_t)ci * 4;
    const int seq = ch[0], t0 = ch[1] + min(warp * WT, ch[2] - 1), n = min(WT, ch[2] - warp * WT), first = p.seq_chunks[seq];
    const bool in = c < p.W;
    Row<VW> zb{}, ub{}, gr[WT];
    WarpGates<VW, TI> g;
    if (in) {
        const TI* gp = (const TI*)p.g + (size_t)t0 * p.ld + c;
#pragma unroll
        for (int t = 0; t < WT; ++t) gr[t] = ld<VW>(gp + (size_t)row_of(t, n) * p.ld);
        if (p.z_b != nullptr) zb = ld<VW>(p.z_b + c);
        if (p.u_b != nullptr) ub = ld<VW>(p.u_b + c);
        g.load(p, c, t0, n, zb, ub);
        // the chunks in front: a warp composes its share of them
        const int per = (ci - first + WARPS - 1) / WARPS, j0 = first + warp * per, j1 = min(ci, j0 + per);
        float2 x[VW];
#pragma unroll
        for (int i = 0; i < VW; ++i) x[i] = make_float2(1.f, 0.f);
#pragma unroll 4
        for (int j = j0; j < j1; ++j)
#pragma unroll
            for (int i = 0; i < VW; ++i) x[i] = then(x[i], p.maps[(size_t)j * p.W + c + i]);
#pragma unroll
        for (int i = 0; i < VW; ++i) {
            before[warp][lane * VW + i] = x[i];
            maps[warp][lane * VW + i] = g.all[i];
        }
    }
    __syncthreads();
    if (!in) return;
    Row<VW> S = ld<VW>(p.start + (size_t)seq * p.W + c);
#pragma unroll
    for (int i = 0; i < VW; ++i) {
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float2 m = before[w][lane * VW + i];
            S.v[i] = m.x * S.v[i] + m.y;
        }
#pragma unroll
        for (int w = 0; w < WARPS - 1; ++w) {
            if (w >= warp) break;
            const float2 m = maps[w][lane * VW + i];
            S.v[i] = m.x * S.v[i] + m.y;
        }
    }
    TO* out = (TO*)p.out + (size_t)t0 * p.ldo + c;
#pragma unroll
    for (int t = 0; t < WT; ++t) {
        if (t >= n) break;
        Row<VW> y;
#pragma unroll
        for (int i = 0; i < VW; ++i) {
            S.v[i] = g.m[t][i].x * S.v[i] + g.m[t][i].y;
            y.v[i] = S.v[i] * (sizeof(TI) == 2 ? silu_fast(gr[t].v[i]) : gr[t].v[i] * sigmoid(gr[t].v[i]));
        }
        st<VW>(out + (size_t)t * p.ldo, y);
    }
    if (ch[3] && n > 0 && (warp + 1) * WT >= ch[2]) st<VW>(p.S + (size_t)p.state_idx[seq] * p.W + c, S);
}

// whole pieces of vw channels everywhere
bool pieces(const MinGruParams* p, int vw, int in_f32, int out_f32) {
    const uintptr_t rows = (uintptr_t)p->z | (uintptr_t)p->u | (uintptr_t)p->g;
    return p->W % vw == 0 && p->ld % vw == 0 && p->ldo % vw == 0 && rows % (vw * (in_f32 ? 4 : 2)) == 0 && (uintptr_t)p->out % (vw * (out_f32 ? 4 : 2)) == 0;
}

}  // namespace

#define SL_BY_TYPE(F, VW)                                        \
    {                                                            \
        if (out_f32) {                                           \
            if (wide) F(VW, float, float) else F(1, float, float) \
        } else if (in_f32) {                                     \
            if (wide) F(VW, float, bf16) else F(1, float, bf16)  \
        } else {                                                 \
            if (wide) F(VW, bf16, bf16) else F(1, bf16, bf16)    \
        }                                                        \
    }

// B sequences, each from its state slot; in_f32 / out_f32: types of the rows and of `out` (fp32 out needs fp32 rows).
SL_API int sl_min_gru_step(const MinGruParams* p, int B, int in_f32, int out_f32, cudaStream_t s) {
    if (B == 0 || p->W == 0) return 0;
    if (B > 65535 || (out_f32 && !in_f32)) return -1;
    const bool wide = pieces(p, 4, in_f32, out_f32);
    const dim3 grid((p->W + (wide ? 511 : 127)) / (wide ? 512 : 128), B);
#define SL_STEP(VW, TI, TO) { sl_launch(min_gru_step_kernel<VW, TI, TO>, grid, 128, 0, s, *p); }
    SL_BY_TYPE(SL_STEP, 4)
#undef SL_STEP
    return SL_LAUNCH_CHECK();
}

// The same over a chunk table that covers every token of the step.
SL_API int sl_min_gru_chunks(const MinGruParams* p, int chunks, int in_f32, int out_f32, cudaStream_t s) {
    if (chunks == 0 || p->W == 0) return 0;
    if (chunks > 65535 || (out_f32 && !in_f32)) return -1;
    const bool wide = pieces(p, 2, in_f32, out_f32);
    const dim3 grid((p->W + (wide ? 63 : 31)) / (wide ? 64 : 32), chunks);
#define SL_CHUNK(VW, TI, TO)                                                \
    {                                                                       \
        sl_launch(min_gru_chunk_kernel<VW, TI>, grid, 256, 0, s, *p);       \
        sl_launch(min_gru_apply_kernel<VW, TI, TO>, grid, 256, 0, s, *p);   \
    }
    SL_BY_TYPE(SL_CHUNK, 2)
#undef SL_CHUNK
    return SL_LAUNCH_CHECK();
}
