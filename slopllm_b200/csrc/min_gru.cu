// minGRU: an element-wise gated recurrence whose gates read the current token only (sm_100a):
//
//   z = sigmoid(z_raw + b_z),  u = u_raw + b_u,  c = u + 1/2 where u >= 0, sigmoid(u) elsewhere
//   S_t = (1 - z_t) S_{t-1} + z_t c_t,   out_t = S_t * silu(g_t)
//
// Gates, candidates, states and their products are fp32; rows and `out` are bf16 or fp32.
//
//  * min_gru_step_kernel: a thread walks a sequence's tokens for VW channels: decoding and short portions, one launch.
//  * min_gru_chunk_kernel, min_gru_apply_kernel: longer portions in chunks of tokens.  A chunk maps the state that enters it to
//    A S + B; the first kernel makes (A, B) of every chunk, the second composes those in front of its own chunk and walks it.
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
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
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
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else {
        r.v[0] = __bfloat162float(*p);
    }
    return r;
}
template <int VW>
__device__ __forceinline__ void st(float* p, const Row<VW>& r) {
    if (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else *p = r.v[0];
}
template <int VW>
__device__ __forceinline__ void st(bf16* p, const Row<VW>& r) {
    if (VW == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162(r.v[0], r.v[1]), f2_to_bf162(r.v[2], r.v[3]));
    else *p = __float2bfloat16(r.v[0]);
}

template <bool FAST>
__device__ __forceinline__ float sigmoid(float x) {
    return FAST ? __fdividef(1.f, 1.f + __expf(-x)) : 1.f / (1.f + expf(-x));
}
// S <- a S + b of one token and channel
template <bool FAST>
__device__ __forceinline__ float2 gate(float z_raw, float u) {
    const float z = sigmoid<FAST>(z_raw), c = u >= 0.f ? u + 0.5f : sigmoid<FAST>(u);
    return make_float2(1.f - z, z * c);
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
            const float2 m = gate<false>(z.v[i] + zb.v[i], u.v[i] + ub.v[i]);
            S.v[i] = m.x * S.v[i] + m.y;
            o.v[i] = S.v[i] * g.v[i] * sigmoid<false>(g.v[i]);
        }
        st<VW>((TO*)p.out + (size_t)t * p.ldo + c, o);
    }
    st<VW>(Sp, S);
}

// grid (ceil(W / (128 * VW)), chunks), block 128
template <int VW, typename TI>
__global__ void __launch_bounds__(128) min_gru_chunk_kernel(MinGruParams p) {
    pdl_grid_sync();
    constexpr bool FAST = sizeof(TI) == 2;
    const int c = (blockIdx.x * 128 + threadIdx.x) * VW;
    const int* ch = p.chunks + (size_t)blockIdx.y * 4;
    const int seq = ch[0], t0 = ch[1], n = ch[2];
    if (c >= p.W) return;
    if ((int)blockIdx.y == p.seq_chunks[seq])                      // (the second kernel overwrites the state while others need it)
        st<VW>(p.start + (size_t)seq * p.W + c, ld<VW>(p.S + (size_t)p.state_idx[seq] * p.W + c));
    if (ch[3]) return;                                             // nobody follows
    Row<VW> zb{}, ub{}, A, B;
    if (p.z_b != nullptr) zb = ld<VW>(p.z_b + c);
    if (p.u_b != nullptr) ub = ld<VW>(p.u_b + c);
#pragma unroll
    for (int i = 0; i < VW; ++i) { A.v[i] = 1.f; B.v[i] = 0.f; }
    const TI *z = (const TI*)p.z + (size_t)t0 * p.ld + c, *u = (const TI*)p.u + (size_t)t0 * p.ld + c;
#pragma unroll 8
    for (int t = 0; t < n; ++t) {
        const Row<VW> zr = ld<VW>(z + (size_t)t * p.ld), ur = ld<VW>(u + (size_t)t * p.ld);
#pragma unroll
        for (int i = 0; i < VW; ++i) {
            const float2 m = gate<FAST>(zr.v[i] + zb.v[i], ur.v[i] + ub.v[i]);
            A.v[i] *= m.x;
            B.v[i] = m.x * B.v[i] + m.y;
        }
    }
    float2* out = p.maps + (size_t)blockIdx.y * p.W + c;
#pragma unroll
    for (int i = 0; i < VW; ++i) out[i] = make_float2(A.v[i], B.v[i]);
}

// grid (ceil(W / (128 * VW)), chunks), block 128; late chunks have most to compose: they start first
template <int VW, typename TI, typename TO>
__global__ void __launch_bounds__(128) min_gru_apply_kernel(MinGruParams p) {
    pdl_grid_sync();
    constexpr bool FAST = sizeof(TI) == 2;
    const int c = (blockIdx.x * 128 + threadIdx.x) * VW, ci = gridDim.y - 1 - blockIdx.y;
    const int* ch = p.chunks + (size_t)ci * 4;
    const int seq = ch[0], t0 = ch[1], n = ch[2];
    if (c >= p.W) return;
    Row<VW> S = ld<VW>(p.start + (size_t)seq * p.W + c), zb{}, ub{};
    if (p.z_b != nullptr) zb = ld<VW>(p.z_b + c);
    if (p.u_b != nullptr) ub = ld<VW>(p.u_b + c);
#pragma unroll 8
    for (int j = p.seq_chunks[seq]; j < ci; ++j) {
        const float2* m = p.maps + (size_t)j * p.W + c;
        if (VW == 4) {
            const Row<4> a = ld<4>(reinterpret_cast<const float*>(m)), b = ld<4>(reinterpret_cast<const float*>(m) + 4);
            S.v[0] = a.v[0] * S.v[0] + a.v[1];
            S.v[VW / 4] = a.v[2] * S.v[VW / 4] + a.v[3];
            S.v[VW / 2] = b.v[0] * S.v[VW / 2] + b.v[1];
            S.v[VW - 1] = b.v[2] * S.v[VW - 1] + b.v[3];
        } else {
            S.v[0] = m->x * S.v[0] + m->y;
        }
    }
    const size_t at = (size_t)t0 * p.ld + c;
    const TI *z = (const TI*)p.z + at, *u = (const TI*)p.u + at, *g = (const TI*)p.g + at;
    TO* out = (TO*)p.out + (size_t)t0 * p.ldo + c;
#pragma unroll 4
    for (int t = 0; t < n; ++t) {
        const size_t o = (size_t)t * p.ld;
        const Row<VW> zr = ld<VW>(z + o), ur = ld<VW>(u + o), gr = ld<VW>(g + o);
        Row<VW> y;
#pragma unroll
        for (int i = 0; i < VW; ++i) {
            const float2 m = gate<FAST>(zr.v[i] + zb.v[i], ur.v[i] + ub.v[i]);
            S.v[i] = m.x * S.v[i] + m.y;
            y.v[i] = S.v[i] * gr.v[i] * sigmoid<FAST>(gr.v[i]);
        }
        st<VW>(out + (size_t)t * p.ldo, y);
    }
    if (ch[3]) st<VW>(p.S + (size_t)p.state_idx[seq] * p.W + c, S);
}

// 16-byte (fp32) or 8-byte (bf16) pieces of four channels everywhere
bool fours(const MinGruParams* p, int in_f32, int out_f32) {
    const uintptr_t rows = (uintptr_t)p->z | (uintptr_t)p->u | (uintptr_t)p->g;
    return p->W % 4 == 0 && p->ld % 4 == 0 && p->ldo % 4 == 0 && rows % (in_f32 ? 16 : 8) == 0 && (uintptr_t)p->out % (out_f32 ? 16 : 8) == 0;
}

}  // namespace

#define SL_BY_TYPE(F)                                       \
    {                                                       \
        if (out_f32) {                                      \
            if (v4) F(4, float, float) else F(1, float, float) \
        } else if (in_f32) {                                \
            if (v4) F(4, float, bf16) else F(1, float, bf16) \
        } else {                                            \
            if (v4) F(4, bf16, bf16) else F(1, bf16, bf16)  \
        }                                                   \
    }

// B sequences, each from its state slot; in_f32 / out_f32: types of the rows and of `out` (fp32 out needs fp32 rows).
SL_API int sl_min_gru_step(const MinGruParams* p, int B, int in_f32, int out_f32, cudaStream_t s) {
    if (B == 0 || p->W == 0) return 0;
    if (B > 65535 || (out_f32 && !in_f32)) return -1;
    const bool v4 = fours(p, in_f32, out_f32);
    const dim3 grid((p->W + (v4 ? 511 : 127)) / (v4 ? 512 : 128), B);
#define SL_STEP(VW, TI, TO) { sl_launch(min_gru_step_kernel<VW, TI, TO>, grid, 128, 0, s, *p); }
    SL_BY_TYPE(SL_STEP)
#undef SL_STEP
    return SL_LAUNCH_CHECK();
}

// The same over a chunk table that covers every token of the step.
SL_API int sl_min_gru_chunks(const MinGruParams* p, int chunks, int in_f32, int out_f32, cudaStream_t s) {
    if (chunks == 0 || p->W == 0) return 0;
    if (chunks > 65535 || (out_f32 && !in_f32)) return -1;
    const bool v4 = fours(p, in_f32, out_f32);
    const dim3 grid((p->W + (v4 ? 511 : 127)) / (v4 ? 512 : 128), chunks);
#define SL_CHUNK(VW, TI, TO)                                                \
    {                                                                       \
        sl_launch(min_gru_chunk_kernel<VW, TI>, grid, 128, 0, s, *p);       \
        sl_launch(min_gru_apply_kernel<VW, TI, TO>, grid, 128, 0, s, *p);   \
    }
    SL_BY_TYPE(SL_CHUNK)
#undef SL_CHUNK
    return SL_LAUNCH_CHECK();
}
