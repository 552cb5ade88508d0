// Residual join, norm and token shift in one pass:
//
//   residual_t = residual_t + y_t            (first call of a step: table[id_t] * scale + places[position_t])
//   h_t        = rms(residual_t) * w
//   out_t      = h_t + (h_{t-1} - h_t) * mix
//
// h_{t-1} of a sequence's first token of the step is the sequence's state (zeros at position 0), and h of its last token becomes it.
//
// A block walks consecutive rows; a thread keeps its columns of the previous row's h in registers.  The row in front of a block's first
// one is made again instead of passed between blocks.  The block of a range's first row also stores the new state: it has read the old
// one by then, in the same threads, so ranges of any length need neither order between blocks nor a second copy of the state.
#include "common.cuh"

namespace {

struct ShiftNormParams {
    void* out; int out_f32;              // [T, H]
    float* res_out;                      // [T, H]
    const float* y; int ldy;             // [T, ldy] (with res_in)
    const float* res_in;                 // [T, H] or null: gathered from `table`
    const long long* ids; const void* table; int table_f32, vocab; float scale;
    const void* places; int num_places;  // [num_places, H] of the table's type, or null
    const float* w;                      // [H]
    const float* mix;                    // [H] or null: no shift
    float* state;                        // [slots, H]
    const int* positions; const int* batch_idx;
    const int* qo;                       // [B + 1]
    const int* slots;                    // [B]
    int H; float eps;
    int* guard;
};

template <int VW>
struct Vec { float v[VW]; };
template <int VW>
__device__ __forceinline__ Vec<VW> ld(const float* p, bool in) {
    Vec<VW> r;
    if (VW == 4) {
        const float4 x = in ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
        r.v[0] = x.x; r.v[VW > 1 ? 1 : 0] = x.y; r.v[VW > 2 ? 2 : 0] = x.z; r.v[VW > 3 ? 3 : 0] = x.w;
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
        r.v[0] = a.x; r.v[VW > 1 ? 1 : 0] = a.y; r.v[VW > 2 ? 2 : 0] = b.x; r.v[VW > 3 ? 3 : 0] = b.y;
    } else {
        r.v[0] = in ? __bfloat162float(*p) : 0.f;
    }
    return r;
}
template <int VW>
__device__ __forceinline__ void st(float* p, const Vec<VW>& x) {
    if (VW == 4) *reinterpret_cast<float4*>(p) = make_float4(x.v[0], x.v[VW > 1 ? 1 : 0], x.v[VW > 2 ? 2 : 0], x.v[VW > 3 ? 3 : 0]);
    else *p = x.v[0];
}
template <int VW>
__device__ __forceinline__ void st(bf16* p, const Vec<VW>& x) {
    if (VW == 4) *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162(x.v[0], x.v[VW > 1 ? 1 : 0]), f2_to_bf162(x.v[VW > 2 ? 2 : 0], x.v[VW > 3 ? 3 : 0]));
    else *p = __float2bfloat16(x.v[0]);
}

// The two addends of a row's columns, loaded a row ahead of their use.
template <int VW, int NV>
struct RowParts { Vec<VW> a[NV], b[NV]; };

template <int VW, int NV, typename TE>
__device__ __forceinline__ void load_row(const ShiftNormParams& p, int t, RowParts<VW, NV>& x) {
    const int tid = threadIdx.x, nt = blockDim.x;
    if (p.res_in != nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (tid + i * nt) * VW;
            x.a[i] = ld<VW>(p.res_in + (size_t)t * p.H + c, c < p.H);
            x.b[i] = ld<VW>(p.y + (size_t)t * p.ldy + c, c < p.H);
        }
        return;
    }
    long long id = p.ids[t];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);              // never read outside the table
    long long at = 0;
    if (p.places != nullptr) {
        at = p.positions[t];
        if (!guard_ok(threadIdx.x == 0 ? p.guard : nullptr, 30, at, p.num_places)) at = 0;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        x.a[i] = ld<VW>((const TE*)p.table + (size_t)id * p.H + c, c < p.H);
        x.b[i] = ld<VW>((const TE*)p.places + (size_t)at * p.H + c, c < p.H && p.places != nullptr);
    }
}

// grid ceil(T / rows); a block takes rows [blockIdx.x * rows, + rows)
template <int VW, int NV, typename TE, typename TO>
__global__ void __launch_bounds__(1024) shift_norm_kernel(ShiftNormParams p, int T, int rows) {
    pdl_grid_sync();
    __shared__ float part[2][32];
    const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, H = p.H;
    const int r0 = blockIdx.x * rows, r1 = min(T, r0 + rows);
    const float scale = p.res_in != nullptr ? 1.f : p.scale;
    Vec<VW> w[NV], mix[NV], prev[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = (tid + i * nt) * VW;
        w[i] = ld<VW>(p.w + c, c < H);
        if (p.mix != nullptr) mix[i] = ld<VW>(p.mix + c, c < H);
#pragma unroll
        for (int j = 0; j < VW; ++j) prev[i].v[j] = 0.f;
    }
    int flip = 0;
    // residual of a row -> x.a, its normed input -> h
    auto norm_row = [&](RowParts<VW, NV>& x, Vec<VW> (&h)[NV]) {
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) {
                x.a[i].v[j] = x.a[i].v[j] * scale + x.b[i].v[j];
                ss += x.a[i].v[j] * x.a[i].v[j];
            }
        ss = warp_sum(ss);
        if (lane == 0) part[flip][warp] = ss;
        __syncthreads();
        ss = 0.f;
        for (int i = 0; i < nt >> 5; ++i) ss += part[flip][i];
        flip ^= 1;                                                    // (the other half was read before this barrier)
        const float inv = 1.f / sqrtf(ss / (float)H + p.eps);
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int j = 0; j < VW; ++j) h[i].v[j] = x.a[i].v[j] * inv * w[i].v[j];
    };
    RowParts<VW, NV> x;
    Vec<VW> h[NV];
    if (p.mix != nullptr && r0 > 0 && p.batch_idx[r0 - 1] == p.batch_idx[r0]) {
        load_row<VW, NV, TE>(p, r0 - 1, x);
        norm_row(x, prev);
    }
    load_row<VW, NV, TE>(p, r0, x);
    for (int t = r0; t < r1; ++t) {
        RowParts<VW, NV> next;
        if (t + 1 < r1) load_row<VW, NV, TE>(p, t + 1, next);
        const int b = p.mix != nullptr ? p.batch_idx[t] : 0;
        const bool first = p.mix != nullptr && t == p.qo[b];
        float* state = first ? p.state + (size_t)p.slots[b] * H : nullptr;
        if (first) {
            const bool fresh = p.positions[t] == 0;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = (tid + i * nt) * VW;
                prev[i] = ld<VW>(state + c, c < H && !fresh);
            }
        }
        norm_row(x, h);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = (tid + i * nt) * VW;
            if (c >= H) continue;
            st<VW>(p.res_out + (size_t)t * H + c, x.a[i]);
            Vec<VW> o = h[i];
            if (p.mix != nullptr)
#pragma unroll
                for (int j = 0; j < VW; ++j) o.v[j] = h[i].v[j] + (prev[i].v[j] - h[i].v[j]) * mix[i].v[j];
            st<VW>((TO*)p.out + (size_t)t * H + c, o);
        }
        if (first) {
            const int last = p.qo[b + 1] - 1;
            if (last != t) {
                RowParts<VW, NV> z;
                load_row<VW, NV, TE>(p, last, z);
                norm_row(z, prev);
            } else {
#pragma unroll
                for (int i = 0; i < NV; ++i) prev[i] = h[i];
            }
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = (tid + i * nt) * VW;
                if (c < H) st<VW>(state + c, prev[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) prev[i] = h[i];
        x = next;
    }
}

template <int VW, typename TE, typename TO>
int run(const ShiftNormParams* p, int T, cudaStream_t s) {
    const int pieces = p->H / VW;
    int nt = (pieces + 31) / 32 * 32;
    if (VW == 4 && nt > 256) nt = (pieces / 2 + 31) / 32 * 32;
    nt = nt < 64 ? 64 : (nt > 1024 ? 1024 : nt);
    const int per = (pieces + nt - 1) / nt;
    const int rows = T <= 296 ? 1 : (T + 591) / 592 < 8 ? (T + 591) / 592 : 8;
    const int blocks = (T + rows - 1) / rows;
#define SL_SN(NV) sl_launch(shift_norm_kernel<VW, NV, TE, TO>, blocks, nt, 0, s, *p, T, rows)
    if (per <= 1) SL_SN(1);
    else if (per <= 2) SL_SN(2);
    else if (per <= 4) SL_SN(4);
    else if (VW == 1) SL_SN(16);                                      // (four values apiece: 4 pieces are 16384 values)
    else return -1;
#undef SL_SN
    return SL_LAUNCH_CHECK();
}

template <typename TE, typename TO>
int run_width(const ShiftNormParams* p, int T, cudaStream_t s) {
    const bool v4 = p->H % 4 == 0 && (p->res_in == nullptr || (p->ldy % 4 == 0 && (uintptr_t)p->y % 16 == 0));
    return v4 ? run<4, TE, TO>(p, T, s) : run<1, TE, TO>(p, T, s);
}

}  // namespace

SL_API int sl_shift_norm(const ShiftNormParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->H < 1 || p->H > 16384 || (p->res_in == nullptr ? p->table == nullptr || p->ids == nullptr : p->y == nullptr)) return -1;
    if (p->positions == nullptr && (p->mix != nullptr || p->places != nullptr)) return -1;
    if (p->mix != nullptr && (p->state == nullptr || p->batch_idx == nullptr || p->qo == nullptr || p->slots == nullptr)) return -1;
    if (p->res_in != nullptr || p->table_f32) return p->out_f32 ? run_width<float, float>(p, T, s) : run_width<float, bf16>(p, T, s);
    return p->out_f32 ? run_width<bf16, float>(p, T, s) : run_width<bf16, bf16>(p, T, s);
}
