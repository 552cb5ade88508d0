// Mixture of small SwiGLU experts with plain (bf16 or fp32) weights.
//
//  * route_softmax_kernel: softmax scores, group-limited choice by corrected scores, a warp per token.
//  * expert_gate_up_kernel, expert_down_kernel: a block takes rows of one expert's matrix and streams them past the tokens that
//    chose the expert, so weights are read once a step and experts that nobody chose are not read at all.
//      - tensor-core form (bf16, rows of whole 16-byte pieces): 16 rows per block, the reduction is split over the warps;
//        operands go from global memory to fragments directly (both sides use the same permutation of the reduction index, so a
//        thread's 16 bytes are two k-steps of its fragment)
//      - plain form: any sizes, fp32 or bf16
//  * expert_sum_kernel: weighted sum of a token's routes, added to its output row; identity experts (ids behind the experts') hand the
//    input through.  identity_experts_kernel adds those alone.
#include "common.cuh"
#include "mma_sync.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu_f(float g) { return g / (1.f + expf(-g)); }

constexpr int MAX_GROUPS = 256, ROUTE_WARPS = 4;

// NPL: experts per lane (E <= 32 * NPL); lane l holds experts l, l + 32, ...
template <int NPL>
__global__ void __launch_bounds__(ROUTE_WARPS * 32) route_softmax_kernel(int* __restrict__ ids, float* __restrict__ wts, const float* __restrict__ logits,
                                                                         int ld, const float* __restrict__ correction, int T, int E, int top, int groups, int keep) {
    pdl_grid_sync();
    __shared__ float best[ROUTE_WARPS][MAX_GROUPS];
    __shared__ bool kept[ROUTE_WARPS][MAX_GROUPS];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * ROUTE_WARPS + warp;
    if (t >= T) return;
    float s[NPL];
    float mx = -INFINITY;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int e = lane + i * 32;
        s[i] = e < E ? logits[(size_t)t * ld + e] : -INFINITY;
        mx = fmaxf(mx, s[i]);
    }
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        s[i] = expf(s[i] - mx);
        sum += s[i];
    }
    const float inv = 1.f / warp_sum(sum);
    const int gsz = E / groups;
#pragma unroll
    for (int i = 0; i < NPL; ++i) s[i] *= inv;
    float c[NPL];                                         // what the choice goes by
#pragma unroll
    for (int i = 0; i < NPL; ++i) c[i] = s[i] + (correction != nullptr && lane + i * 32 < E ? correction[lane + i * 32] : 0.f);
    if (groups > 1) {
        for (int g = lane; g < groups; g += 32) best[warp][g] = -INFINITY;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NPL; ++i) {
            const int e = lane + i * 32;
            if (e >= E) continue;
            // (the order of numbers from zero up is that of their bits, below zero the reverse of it)
            if (c[i] >= 0.f) atomicMax(reinterpret_cast<int*>(&best[warp][e / gsz]), __float_as_int(c[i] + 0.f));
            else atomicMin(reinterpret_cast<unsigned*>(&best[warp][e / gsz]), __float_as_uint(c[i]));
        }
        __syncwarp();
        for (int g = lane; g < groups; g += 32) {
            int beaten = 0;
            for (int o = 0; o < groups; ++o) beaten += best[warp][o] > best[warp][g] || (best[warp][o] == best[warp][g] && o < g);
            kept[warp][g] = beaten < keep;
        }
        __syncwarp();
    }
    unsigned taken = 0;                                   // bit i: expert lane + 32 i is out
#pragma unroll
    for (int i = 0; i < NPL; ++i) {
        const int e = lane + i * 32;
        if (e >= E || (groups > 1 && !kept[warp][e / gsz])) taken |= 1u << i;
    }
    for (int r = 0; r < top; ++r) {
        float v = -INFINITY, weight = 0.f;
        int id = 0x7fffffff, mine = 0;
#pragma unroll
        for (int i = 0; i < NPL; ++i)
            if (!((taken >> i) & 1u) && c[i] > v) { v = c[i]; weight = s[i]; id = lane + i * 32; mine = i; }
        const int my_id = id;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, v, o);
            const int oid = __shfl_xor_sync(0xffffffffu, id, o);
            if (ov > v || (ov == v && oid < id)) { v = ov; id = oid; }
        }
        if (my_id == id && id < E) {                      // (one lane: ids differ between the lanes)
            taken |= 1u << mine;
            ids[(size_t)t * top + r] = id;
            wts[(size_t)t * top + r] = weight;
        } else if (id >= E && lane == 0) {                // (logits that are no numbers)
            ids[(size_t)t * top + r] = 0;
            wts[(size_t)t * top + r] = 0.f;
        }
    }
}

struct ExpertStreamParams {
    const void* x; int ldx;              // [T, ldx]
    const int* ids; const float* wts;    // [T, top]
    int T, top, H, I, E;
    const void *w13, *w2;                // [E, 2I, H] (gate | up), [E, H, I]
    void* act;                           // [T * top, I]
    float* y_route;                      // [T * top, H]
    float* out; int ldo;                 // [T, ldo], added to
    int identity;                        // ids from E on: the input times the weight is added (else nothing)
};

constexpr int LIST = 1024;               // routes looked through at a time

// The routes among [r0, r0 + LIST) that chose expert e, in ascending order.  All 256 threads; the list is valid after it returns.
__device__ __forceinline__ int find_routes(const ExpertStreamParams& p, int e, int r0, short* list, int* counts) {
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = min(LIST, p.T * p.top - r0);
    __syncthreads();
    unsigned hit[LIST / 256];
#pragma unroll
    for (int i = 0; i < LIST / 256; ++i) {               // warp w looks at routes [128 w, 128 w + 128)
        const int j = warp * (LIST / 8) + i * 32 + lane;
        hit[i] = __ballot_sync(0xffffffffu, j < n && p.ids[r0 + j] == e);
    }
    if (lane == 0) {
        int c = 0;
#pragma unroll
        for (int i = 0; i < LIST / 256; ++i) c += __popc(hit[i]);
        counts[warp] = c;
    }
    __syncthreads();
    int at = 0, total = 0;
    for (int w = 0; w < 8; ++w) {
        if (w < warp) at += counts[w];
        total += counts[w];
    }
#pragma unroll
    for (int i = 0; i < LIST / 256; ++i) {
        if ((hit[i] >> lane) & 1u) list[at + __popc(hit[i] & ((1u << lane) - 1u))] = (short)(warp * (LIST / 8) + i * 32 + lane);
        at += __popc(hit[i]);
    }
    __syncthreads();
    return total;
}

// ---- plain form: a warp per matrix row; grid (ceil(rows / 8), E), block 256 ----
template <typename T>
__global__ void __launch_bounds__(256) expert_gate_up_plain_kernel(ExpertStreamParams p) {
    pdl_grid_sync();
    __shared__ short list[LIST];
    __shared__ int counts[8];
    const int e = blockIdx.y, lane = threadIdx.x & 31, n = blockIdx.x * 8 + (threadIdx.x >> 5);
    const T *wg = (const T*)p.w13 + ((size_t)e * 2 * p.I + n) * p.H, *wu = wg + (size_t)p.I * p.H;
    for (int r0 = 0; r0 < p.T * p.top; r0 += LIST) {
        const int cnt = find_routes(p, e, r0, list, counts);
        if (n >= p.I) continue;
        for (int j = 0; j < cnt; ++j) {
            const int route = r0 + list[j];
            const T* x = (const T*)p.x + (size_t)(route / p.top) * p.ldx;
            float a = 0.f, b = 0.f;
            for (int i = lane; i < p.H; i += 32) {
                const float v = to_f(x[i]);
                a += to_f(wg[i]) * v;
                b += to_f(wu[i]) * v;
            }
            a = warp_sum(a);
            b = warp_sum(b);
            if (lane == 0) put((T*)p.act + (size_t)route * p.I + n, silu_f(a) * b);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) expert_down_plain_kernel(ExpertStreamParams p) {
    pdl_grid_sync();
    __shared__ short list[LIST];
    __shared__ int counts[8];
    const int e = blockIdx.y, lane = threadIdx.x & 31, n = blockIdx.x * 8 + (threadIdx.x >> 5);
    const T* w = (const T*)p.w2 + ((size_t)e * p.H + n) * p.I;
    for (int r0 = 0; r0 < p.T * p.top; r0 += LIST) {
        const int cnt = find_routes(p, e, r0, list, counts);
        if (n >= p.H) continue;
        for (int j = 0; j < cnt; ++j) {
            const int route = r0 + list[j];
            const T* x = (const T*)p.act + (size_t)route * p.I;
            float a = 0.f;
            for (int i = lane; i < p.I; i += 32) a += to_f(w[i]) * to_f(x[i]);
            a = warp_sum(a);
            if (lane == 0) p.y_route[(size_t)route * p.H + n] = a;
        }
    }
}

// ---- tensor-core form: 16 rows (of gate and of up, or of down) per block, eight warps share the reduction ----
constexpr int ROWS = 16;

// sum_k w[row, k] x[n, k] over the warp's share of K for MT row tiles (16 rows each, `tile_stride` elements apart) and NT token
// tiles of 8.  w: first row; xr[i]: row of token tile i's token g (lane >> 2).
template <int MT, int NT>
__device__ __forceinline__ void stream_tile(float (&acc)[MT][NT][4], const bf16* w, size_t tile_stride, const bf16* const (&xr)[NT], int K, int warp) {
    const int lane = threadIdx.x & 31, g = lane >> 2, c4 = lane & 3;
    const bf16* wr = w + (size_t)g * K + c4 * 8;
    const size_t half = (size_t)8 * K;
    constexpr int U = MT * NT <= 2 ? 4 : 2;
    for (int k0 = warp * 32; k0 < K; k0 += 256 * U) {
        uint4 a[U][MT][2], b[U][NT];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int k = k0 + u * 256;
            const bool in = k + c4 * 8 < K;                        // (K % 8 == 0; the last 32 may be ragged)
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                a[u][m][0] = in ? ldg_nc_16(wr + m * tile_stride + k) : make_uint4(0, 0, 0, 0);
                a[u][m][1] = in ? ldg_nc_16(wr + m * tile_stride + half + k) : make_uint4(0, 0, 0, 0);
            }
#pragma unroll
            for (int n = 0; n < NT; ++n)
                b[u][n] = in && xr[n] != nullptr ? *reinterpret_cast<const uint4*>(xr[n] + k + c4 * 8) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
        for (int u = 0; u < U; ++u)
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const uint32_t s0[4] = {a[u][m][0].x, a[u][m][1].x, a[u][m][0].y, a[u][m][1].y};
                const uint32_t s1[4] = {a[u][m][0].z, a[u][m][1].z, a[u][m][0].w, a[u][m][1].w};
#pragma unroll
                for (int n = 0; n < NT; ++n) {
                    mma_bf16_16816(acc[m][n], s0, b[u][n].x, b[u][n].y);
                    mma_bf16_16816(acc[m][n], s1, b[u][n].z, b[u][n].w);
                }
            }
    }
}

// grid (rows / ROWS, E), block 256.  GATE_UP: act = silu(gate) * up; otherwise y_route = down.
template <bool GATE_UP, int NT>
__global__ void __launch_bounds__(256) expert_mma_kernel(ExpertStreamParams p) {
    pdl_grid_sync();
    constexpr int MT = GATE_UP ? 2 : 1;
    __shared__ short list[LIST];
    __shared__ int counts[8];
    __shared__ float red[8][MT * ROWS][NT * 8 + 1];
    const int e = blockIdx.y, n0 = blockIdx.x * ROWS, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int K = GATE_UP ? p.H : p.I, N = GATE_UP ? p.I : p.H;
    const bf16* w = GATE_UP ? (const bf16*)p.w13 + ((size_t)e * 2 * p.I + n0) * p.H : (const bf16*)p.w2 + ((size_t)e * p.H + n0) * p.I;
    for (int r0 = 0; r0 < p.T * p.top; r0 += LIST) {
        const int cnt = find_routes(p, e, r0, list, counts);
        for (int j0 = 0; j0 < cnt; j0 += NT * 8) {
            const bf16* xr[NT];
#pragma unroll
            for (int i = 0; i < NT; ++i) {
                const int j = j0 + i * 8 + g;
                xr[i] = nullptr;
                if (j < cnt) {
                    const int route = r0 + list[j];
                    xr[i] = GATE_UP ? (const bf16*)p.x + (size_t)(route / p.top) * p.ldx : (const bf16*)p.act + (size_t)route * p.I;
                }
            }
            float acc[MT][NT][4] = {};
            stream_tile<MT, NT>(acc, w, (size_t)p.I * p.H, xr, K, warp);
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int i = 0; i < NT; ++i) {
                    float *a = &red[warp][m * ROWS + g][i * 8 + c4 * 2], *b = &red[warp][m * ROWS + g + 8][i * 8 + c4 * 2];
                    a[0] = acc[m][i][0]; a[1] = acc[m][i][1];
                    b[0] = acc[m][i][2]; b[1] = acc[m][i][3];
                }
            __syncthreads();
            for (int i = tid; i < ROWS * NT * 8; i += 256) {
                const int n = i % ROWS, j = i / ROWS;
                if (j0 + j >= cnt || n0 + n >= N) continue;
                const int route = r0 + list[j0 + j];
                float s = 0.f, u = 0.f;
#pragma unroll
                for (int x = 0; x < 8; ++x) {
                    s += red[x][n][j];
                    if (GATE_UP) u += red[x][(MT - 1) * ROWS + n][j];
                }
                if (GATE_UP) ((bf16*)p.act)[(size_t)route * p.I + n0 + n] = __float2bfloat16(silu_f(s) * u);
                else p.y_route[(size_t)route * p.H + n0 + n] = s;
            }
            __syncthreads();
        }
    }
}

// grid (ceil(H / 256), T)
template <typename T>
__global__ void __launch_bounds__(256) expert_sum_kernel(ExpertStreamParams p) {
    pdl_grid_sync();
    const int n = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (n >= p.H) return;
    float a = p.out[(size_t)t * p.ldo + n];
#pragma unroll 8
    for (int j = 0; j < p.top; ++j) {
        const float w = p.wts[t * p.top + j];
        if (p.ids[t * p.top + j] < p.E) a += w * p.y_route[((size_t)t * p.top + j) * p.H + n];
        else if (p.identity) a += w * to_f(((const T*)p.x)[(size_t)t * p.ldx + n]);
    }
    p.out[(size_t)t * p.ldo + n] = a;
}

// out[t] += x[t] * sum of the weights of t's identity experts.  grid (ceil(H / (256 VW)), T)
template <int VW, typename T>
__global__ void __launch_bounds__(256) identity_experts_kernel(float* __restrict__ out, int ldo, const T* __restrict__ x, int ldx, const int* __restrict__ ids,
                                                               const float* __restrict__ wts, int top, int H, int E) {
    pdl_grid_sync();
    const int n = (blockIdx.x * 256 + threadIdx.x) * VW, t = blockIdx.y;
    if (n >= H) return;
    float w = 0.f;
    for (int j = 0; j < top; ++j) w += ids[t * top + j] >= E ? wts[t * top + j] : 0.f;
    if (w == 0.f) return;
    float* o = out + (size_t)t * ldo + n;
    const T* v = x + (size_t)t * ldx + n;
    if (VW == 4) {
        const uint2 u = *reinterpret_cast<const uint2*>(v);           // (bf16 only)
        const float2 a = bf162_to_f2(u.x), b = bf162_to_f2(u.y);
        float4 r = *reinterpret_cast<float4*>(o);
        r.x += w * a.x; r.y += w * a.y; r.z += w * b.x; r.w += w * b.y;
        *reinterpret_cast<float4*>(o) = r;
    } else {
        *o += w * to_f(*v);
    }
}

}  // namespace

// logits fp32 [T, ld]; correction fp32 [E] or null.  E <= 1024, groups <= 256 equal runs, top <= experts of the kept groups.
SL_API int sl_route_softmax(void* ids, void* wts, const void* logits, int ld, const void* correction, int T, int E, int top, int groups, int keep, cudaStream_t s) {
    if (T == 0) return 0;
    if (E < 1 || E > 1024 || groups < 1 || groups > MAX_GROUPS || E % groups != 0 || keep < 1 || keep > groups || top < 1 || top > keep * (E / groups)) return -1;
    const int blocks = (T + ROUTE_WARPS - 1) / ROUTE_WARPS;
#define SL_RS(N) sl_launch(route_softmax_kernel<N>, blocks, ROUTE_WARPS * 32, 0, s, (int*)ids, (float*)wts, (const float*)logits, ld, (const float*)correction, T, E, top, groups, keep)
    if (E <= 32) SL_RS(1);
    else if (E <= 64) SL_RS(2);
    else if (E <= 128) SL_RS(4);
    else if (E <= 256) SL_RS(8);
    else if (E <= 512) SL_RS(16);
    else SL_RS(32);
#undef SL_RS
    return SL_LAUNCH_CHECK();
}

// f32: x, weights and act are fp32 (else bf16).
SL_API int sl_expert_stream(const ExpertStreamParams* p, int f32, cudaStream_t s) {
    if (p->T == 0) return 0;
    if (p->E < 1 || p->E > 65535 || p->T > 65535 || p->top < 1) return -1;
    const bool mma = !f32 && p->H % ROWS == 0 && p->I % ROWS == 0 && p->ldx % 8 == 0 && ((uintptr_t)p->x | (uintptr_t)p->w13 | (uintptr_t)p->w2) % 16 == 0;
    if (mma) {
        if (p->T * p->top <= 8 * p->E) {
            sl_launch(expert_mma_kernel<true, 1>, dim3(p->I / ROWS, p->E), 256, 0, s, *p);
            sl_launch(expert_mma_kernel<false, 1>, dim3(p->H / ROWS, p->E), 256, 0, s, *p);
        } else {
            sl_launch(expert_mma_kernel<true, 2>, dim3(p->I / ROWS, p->E), 256, 0, s, *p);
            sl_launch(expert_mma_kernel<false, 2>, dim3(p->H / ROWS, p->E), 256, 0, s, *p);
        }
    } else if (f32) {
        sl_launch(expert_gate_up_plain_kernel<float>, dim3((p->I + 7) / 8, p->E), 256, 0, s, *p);
        sl_launch(expert_down_plain_kernel<float>, dim3((p->H + 7) / 8, p->E), 256, 0, s, *p);
    } else {
        sl_launch(expert_gate_up_plain_kernel<bf16>, dim3((p->I + 7) / 8, p->E), 256, 0, s, *p);
        sl_launch(expert_down_plain_kernel<bf16>, dim3((p->H + 7) / 8, p->E), 256, 0, s, *p);
    }
    if (f32) sl_launch(expert_sum_kernel<float>, dim3((p->H + 255) / 256, p->T), 256, 0, s, *p);
    else sl_launch(expert_sum_kernel<bf16>, dim3((p->H + 255) / 256, p->T), 256, 0, s, *p);
    return SL_LAUNCH_CHECK();
}

// out fp32 [T, ldo] += x [T, ldx] times the weights of the routes (ids, wts [T, top]) whose id is E or more
SL_API int sl_identity_experts(float* out, int ldo, const void* x, int ldx, const int* ids, const float* wts, int T, int top, int H, int E, int f32,
                               cudaStream_t s) {
    if (T == 0) return 0;
    if (T > 65535) return -1;
    const bool v4 = !f32 && H % 4 == 0 && ldo % 4 == 0 && ldx % 4 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)x % 8 == 0;
    if (f32) sl_launch(identity_experts_kernel<1, float>, dim3((H + 255) / 256, T), 256, 0, s, out, ldo, (const float*)x, ldx, ids, wts, top, H, E);
    else if (v4) sl_launch(identity_experts_kernel<4, bf16>, dim3((H / 4 + 255) / 256, T), 256, 0, s, out, ldo, (const bf16*)x, ldx, ids, wts, top, H, E);
    else sl_launch(identity_experts_kernel<1, bf16>, dim3((H + 255) / 256, T), 256, 0, s, out, ldo, (const bf16*)x, ldx, ids, wts, top, H, E);
    return SL_LAUNCH_CHECK();
}
