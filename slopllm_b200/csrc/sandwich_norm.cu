// Residual stream of decoders that normalise a sublayer's output before it is added ("sandwich" norms):
//
//   residual' = residual + rms(y) * w_post          (y: the sublayer's output, fp32; absent in front of the first sublayer;
//                                                    without w_post it is added as it is)
//   out       = rms(residual') * w_next             (input of the next sublayer, or of the output head)
//
// and of decoders that normalise the sum instead ("post" norms): x is the residual itself,
//
//   x'  = rms(alpha * x + y + bias) * w             (without y, as in front of the first sublayer: x' = x)
//   out = x', or rms(x') * w_next                   (input of the next sublayer, of the output head)
//
// in one pass over the token's row, which stays in registers between the two reductions.  The first call of a step gathers
// the residual from the embedding table instead.  Weights, sums and the residual are fp32; `out` is bf16 or fp32.
#include "common.cuh"

namespace {

struct PostNormParams {
    void* out; int out_f32;          // [T, H]
    float* res_out;                  // [T, H]
    const float* y; int ldy;         // [T, ldy] or null
    const float* w_post;             // [H] or null (with y)
    const float* res_in;             // [T, H] or null: gathered from `table`
    const long long* ids; const void* table; int table_f32, vocab;
    const float* w_next;             // [H]
    int H; float eps;
};

// Sum over the block with one barrier; `part` is used once per kernel.
__device__ __forceinline__ float one_barrier_sum(float v, float* part) {
    const int nw = blockDim.x >> 5;
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
    for (int i = 0; i < nw; ++i) s += part[i];
    return s;
}

template <int VW>
struct Vec { float v[VW]; };
template <int VW>
__device__ __forceinline__ Vec<VW> ld(const float* p, bool in) {
    Vec<VW> r;
    if (VW == 4) {
        const float4 x = in ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
        r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w;
    } else {
        r.v[0] = in ? *p : 0.f;
    }
    return r;
}
template <int VW>
__device__ __forceinline__ Vec<VW> ld(const bf16* p, bool in) {
    Vec<VW> r;
    if (VW == 4) {
        const uint2 x = in ? *reinterpret_cast<const uint2*>(p) : make_uint2(0, 0);
        const float2 a = bf162_to_f2(x.x), b = bf162_to_f2(x.y);
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else {
        r.v[0] = in ? __bfloat162float(*p) : 0.f;
    }
    return r;
}
template <int VW>
__device__ __forceinline__ void st(float* p, const float* v) {
    if (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    else *p = v[0];
}
template <int VW>
__device__ __forceinline__ void st(bf16* p, const float* v) {
    if (VW == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162(v[0], v[1]), f2_to_bf162(v[2], v[3]));
    else *p = __float2bfloat16(v[0]);
}

// One block per token; a thread holds NV pieces of VW values, all of whose loads are issued before the first reduction.
template <int VW, int NV>
__global__ void __launch_bounds__(1024) post_norm_kernel(PostNormParams p) {
    pdl_grid_sync();
    __shared__ float part[2][32];
    const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, H = p.H;
    Vec<VW> r[NV], y[NV], wp[NV], wn[NV];
    long long id = 0;
    if (p.res_in == nullptr) {
        id = p.ids[t];
        id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);      // never read outside the table
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        const bool in = c < H;
        if (p.res_in != nullptr) r[i] = ld<VW>(p.res_in + (size_t)t * H + c, in);
        else if (p.table_f32) r[i] = ld<VW>((const float*)p.table + (size_t)id * H + c, in);
        else r[i] = ld<VW>((const bf16*)p.table + (size_t)id * H + c, in);
        wn[i] = ld<VW>(p.w_next + c, in);
        if (p.y != nullptr) {
            y[i] = ld<VW>(p.y + (size_t)t * p.ldy + c, in);
            if (p.w_post != nullptr) wp[i] = ld<VW>(p.w_post + c, in);
        }
    }
    if (p.y != nullptr && p.w_post == nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) r[i].v[j] += y[i].v[j];
    } else if (p.y != nullptr) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) ss += y[i].v[j] * y[i].v[j];
        const float inv = 1.f / sqrtf(one_barrier_sum(ss, part[0]) / (float)H + p.eps);
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) r[i].v[j] += y[i].v[j] * inv * wp[i].v[j];
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i)
#pragma unroll
        for (int j = 0; j < VW; ++j) ss += r[i].v[j] * r[i].v[j];
    const float inv = 1.f / sqrtf(one_barrier_sum(ss, part[1]) / (float)H + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= H) continue;
        st<VW>(p.res_out + (size_t)t * H + c, r[i].v);
        float o[VW];
#pragma unroll
        for (int j = 0; j < VW; ++j) o[j] = r[i].v[j] * inv * wn[i].v[j];
        if (p.out_f32) st<VW>((float*)p.out + (size_t)t * H + c, o);
        else st<VW>((bf16*)p.out + (size_t)t * H + c, o);
    }
}

struct SumNormParams {
    void* out; int out_f32;          // [T, H]
    float* res_out;                  // [T, H]: x'
    const float* y; int ldy;         // [T, ldy] or null
    const float* bias;               // [H] or null
    float alpha;
    const float* w;                  // [H] (with y)
    const float* res_in;             // [T, H] or null: gathered from `table`
    const long long* ids; const void* table; int table_f32, vocab;
    const float* w_next;             // [H] or null
    int H; float eps;
};

template <int VW, int NV>
__global__ void __launch_bounds__(1024) sum_norm_kernel(SumNormParams p) {
    pdl_grid_sync();
    __shared__ float part[2][32];
    const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, H = p.H;
    Vec<VW> r[NV], y[NV], w[NV], wn[NV];
    long long id = 0;
    if (p.res_in == nullptr) {
        id = p.ids[t];
        id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);      // never read outside the table
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        const bool in = c < H;
        if (p.res_in != nullptr) r[i] = ld<VW>(p.res_in + (size_t)t * H + c, in);
        else if (p.table_f32) r[i] = ld<VW>((const float*)p.table + (size_t)id * H + c, in);
        else r[i] = ld<VW>((const bf16*)p.table + (size_t)id * H + c, in);
        if (p.w_next != nullptr) wn[i] = ld<VW>(p.w_next + c, in);
        if (p.y != nullptr) {
            y[i] = ld<VW>(p.y + (size_t)t * p.ldy + c, in);
            w[i] = ld<VW>(p.w + c, in);
            if (p.bias != nullptr) {
                const Vec<VW> b = ld<VW>(p.bias + c, in);
#pragma unroll
                for (int j = 0; j < VW; ++j) y[i].v[j] += b.v[j];
            }
        }
    }
    auto inverse_rms = [&](float* buf) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) ss += r[i].v[j] * r[i].v[j];
        return 1.f / sqrtf(one_barrier_sum(ss, buf) / (float)H + p.eps);
    };
    if (p.y != nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) r[i].v[j] = p.alpha * r[i].v[j] + y[i].v[j];
        const float inv = inverse_rms(part[0]);
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) r[i].v[j] *= inv * w[i].v[j];
    }
    const float inv = p.w_next != nullptr ? inverse_rms(part[1]) : 1.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        if (c >= H) continue;
        st<VW>(p.res_out + (size_t)t * H + c, r[i].v);
        float o[VW];
#pragma unroll
        for (int j = 0; j < VW; ++j) o[j] = p.w_next != nullptr ? r[i].v[j] * inv * wn[i].v[j] : r[i].v[j];
        if (p.out_f32) st<VW>((float*)p.out + (size_t)t * H + c, o);
        else st<VW>((bf16*)p.out + (size_t)t * H + c, o);
    }
}

// Threads of a block and pieces of VW values per thread for a row of H values.
void row_split(int H, int VW, int& nt, int& per) {
    const int pieces = H / VW;
    nt = (pieces + 31) / 32 * 32;
    if (VW == 4 && nt > 256) nt = (pieces / 2 + 31) / 32 * 32;       // two pieces per thread
    nt = nt < 64 ? 64 : (nt > 1024 ? 1024 : nt);
    per = (pieces + nt - 1) / nt;
}

template <int VW>
int launch_sum_norm(const SumNormParams* p, int T, cudaStream_t s) {
    int nt, per;
    row_split(p->H, VW, nt, per);
    if (per <= 1) sl_launch(sum_norm_kernel<VW, 1>, T, nt, 0, s, *p);
    else if (per <= 2) sl_launch(sum_norm_kernel<VW, 2>, T, nt, 0, s, *p);
    else if (per <= 4) sl_launch(sum_norm_kernel<VW, 4>, T, nt, 0, s, *p);
    else if (VW == 1) sl_launch(sum_norm_kernel<1, 16>, T, nt, 0, s, *p);      // (four values apiece: 4 pieces are 16384 values)
    else return -1;
    return SL_LAUNCH_CHECK();
}

template <int VW>
int launch_post_norm(const PostNormParams* p, int T, cudaStream_t s) {
    int nt, per;
    row_split(p->H, VW, nt, per);
    if (per <= 1) sl_launch(post_norm_kernel<VW, 1>, T, nt, 0, s, *p);
    else if (per <= 2) sl_launch(post_norm_kernel<VW, 2>, T, nt, 0, s, *p);
    else if (per <= 4) sl_launch(post_norm_kernel<VW, 4>, T, nt, 0, s, *p);
    else sl_launch(post_norm_kernel<VW, 16>, T, nt, 0, s, *p);
    return SL_LAUNCH_CHECK();
}

}  // namespace

SL_API int sl_post_norm(const PostNormParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->H < 1 || p->H > 16384 || (p->res_in == nullptr && p->table == nullptr)) return -1;
    const bool v4 = p->H % 4 == 0 && (p->y == nullptr || (p->ldy % 4 == 0 && (uintptr_t)p->y % 16 == 0));
    return v4 ? launch_post_norm<4>(p, T, s) : launch_post_norm<1>(p, T, s);
}

SL_API int sl_sum_norm(const SumNormParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->H < 1 || p->H > 16384 || (p->res_in == nullptr && p->table == nullptr) || (p->y != nullptr && p->w == nullptr)) return -1;
    const bool v4 = p->H % 4 == 0 && (p->y == nullptr || (p->ldy % 4 == 0 && (uintptr_t)p->y % 16 == 0));
    return v4 ? launch_sum_norm<4>(p, T, s) : launch_sum_norm<1>(p, T, s);
}
