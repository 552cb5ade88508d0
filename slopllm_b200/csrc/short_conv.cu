// Depthwise causal convolution over time with silu, parallel over tokens:
//
//   y[t, c] = silu(sum_j w[j, c] x[t - (taps-1) + j, c])
//
// Inputs before the token range of a sequence come from its ring, state[slot][p % taps][c] = input of position p (zeros before
// the start).  The block of a range's first tokens also stores the range's last inputs: a thread reads what it needs of its
// channel before it overwrites it, and no other block touches the ring, so one launch suffices.
#include "common.cuh"

namespace {

constexpr int CHUNK = 32;        // tokens per block

template <int V>
struct Vals { float v[V]; };
template <int V>
__device__ __forceinline__ Vals<V> load(const float* p) {
    Vals<V> r;
    if (V == 2) { const float2 x = *reinterpret_cast<const float2*>(p); r.v[0] = x.x; r.v[V - 1] = x.y; }
    else r.v[0] = *p;
    return r;
}
template <int V>
__device__ __forceinline__ Vals<V> load(const bf16* p) {
    Vals<V> r;
    if (V == 2) { const float2 x = bf162_to_f2(*reinterpret_cast<const uint32_t*>(p)); r.v[0] = x.x; r.v[V - 1] = x.y; }
    else r.v[0] = __bfloat162float(*p);
    return r;
}
template <int V>
__device__ __forceinline__ void store(float* p, const Vals<V>& x) {
    if (V == 2) *reinterpret_cast<float2*>(p) = make_float2(x.v[0], x.v[V - 1]);
    else *p = x.v[0];
}
template <int V>
__device__ __forceinline__ void store(bf16* p, const Vals<V>& x) {
    if (V == 2) *reinterpret_cast<uint32_t*>(p) = f2_to_bf162(x.v[0], x.v[V - 1]);
    else *p = __float2bfloat16(x.v[0]);
}

// grid (ceil(C / (128 * V)), ceil(longest / CHUNK), B), block 128: V channels per thread.  taps <= MAXT.
template <int MAXT, int V, typename TI, typename TO>
__global__ void __launch_bounds__(128) short_conv_kernel(TO* __restrict__ y, const TI* __restrict__ x, int ldx, const float* __restrict__ w,
                                                         float* __restrict__ state, const int* __restrict__ positions,
                                                         const int* __restrict__ qo_indptr, const int* __restrict__ state_idx, int C, int taps) {
    pdl_grid_sync();
    const int c = (blockIdx.x * 128 + threadIdx.x) * V, seq = blockIdx.z;
    const int lo = qo_indptr[seq], hi = qo_indptr[seq + 1], t0 = lo + blockIdx.y * CHUNK, t1 = min(hi, t0 + CHUNK);
    if (c >= C || t0 >= t1) return;
    float* ring = state + (size_t)state_idx[seq] * taps * C + c;
    const int start = positions[lo];
    Vals<V> win[MAXT], wt[MAXT], zero;
#pragma unroll
    for (int u = 0; u < V; ++u) zero.v[u] = 0.f;
#pragma unroll
    for (int j = 0; j < MAXT; ++j) {
        wt[j] = j < taps ? load<V>(w + (size_t)j * C + c) : zero;
        win[j] = zero;
        const int t = t0 - (taps - 1) + j;                         // win[j] is the input of token t
        if (j < taps - 1) {
            const int p = start + t - lo;
            if (t >= lo) win[j] = load<V>(x + (size_t)t * ldx + c);
            else if (p >= 0) win[j] = load<V>(ring + (size_t)(p % taps) * C);
        }
    }
    for (int t = t0; t < t1; t += 8) {
        Vals<V> in[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) in[i] = t + i < t1 ? load<V>(x + (size_t)(t + i) * ldx + c) : zero;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (t + i >= t1) break;
            Vals<V> a = zero;
#pragma unroll
            for (int j = 0; j < MAXT; ++j) {
                if (j == taps - 1) win[j] = in[i];
#pragma unroll
                for (int u = 0; u < V; ++u) a.v[u] += wt[j].v[u] * win[j].v[u];
            }
#pragma unroll
            for (int u = 0; u < V; ++u) a.v[u] = sizeof(TO) == 2 ? __fdividef(a.v[u], 1.f + __expf(-a.v[u])) : a.v[u] / (1.f + expf(-a.v[u]));
            store<V>(y + (size_t)(t + i) * C + c, a);
#pragma unroll
            for (int j = 0; j + 1 < MAXT; ++j) win[j] = win[j + 1];
        }
    }
    if (blockIdx.y == 0)
        for (int t = max(lo, hi - taps); t < hi; ++t) store<V>(ring + (size_t)((start + t - lo) % taps) * C, load<V>(x + (size_t)t * ldx + c));
}

}  // namespace

// y [T, C], x [T, ldx], w fp32 [taps, C], state fp32 [slots, taps, C].
SL_API int sl_short_conv(void* y, const void* x, int ldx, const void* w, void* state, const void* positions, const void* qo_indptr,
                         const void* state_idx, int B, int longest, int C, int taps, int in_f32, int out_f32, cudaStream_t s) {
    if (B == 0 || longest == 0 || C == 0) return 0;
    if (taps < 1 || taps > 16 || B > 65535 || (longest + CHUNK - 1) / CHUNK > 65535 || (out_f32 && !in_f32)) return -1;
    const bool pairs = C % 2 == 0 && ldx % 2 == 0 && (uintptr_t)x % 8 == 0;
    const dim3 grid((C + (pairs ? 255 : 127)) / (pairs ? 256 : 128), (longest + CHUNK - 1) / CHUNK, B);
#define SL_CONV(M, V, TI, TO)                                                                                                         \
    sl_launch(short_conv_kernel<M, V, TI, TO>, grid, 128, 0, s, (TO*)y, (const TI*)x, ldx, (const float*)w, (float*)state, (const int*)positions, \
              (const int*)qo_indptr, (const int*)state_idx, C, taps)
#define SL_CONV_T(M, V)                                \
    {                                                  \
        if (out_f32) SL_CONV(M, V, float, float);      \
        else if (in_f32) SL_CONV(M, V, float, bf16);   \
        else SL_CONV(M, V, bf16, bf16);                \
    }
    if (taps <= 4 && pairs) SL_CONV_T(4, 2) else if (taps <= 4) SL_CONV_T(4, 1) else if (taps <= 8 && pairs) SL_CONV_T(8, 2)
    else if (taps <= 8) SL_CONV_T(8, 1) else if (pairs) SL_CONV_T(16, 2) else SL_CONV_T(16, 1)
#undef SL_CONV_T
#undef SL_CONV
    return SL_LAUNCH_CHECK();
}
