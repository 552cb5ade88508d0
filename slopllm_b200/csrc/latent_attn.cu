// Latent attention over a paged cache of plain (bf16 or fp32) rows [latent | rotated key part], shared by all heads, with a
// sliding window and a softmax sink.
//
//  * latent_pre_kernel: RMS norm of the latent, rotary (rotate-half, any frequency table) of the shared key part and of the
//    heads' rotated query parts; the cache row is written straight into its slot.
//  * latent_rows_kernel: absorbed attention (query rows already multiplied by W_uk) of independent token rows on the CUDA
//    cores, any sizes, bf16 or fp32.
#include "common.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

struct LatentPreParams {
    const void* qd; int ld;              // [T, ld]: heads x (dim | rot_dim), then latent (rank), then shared key part (rot_dim)
    int heads, dim, rot_dim, rot_dims, rank;
    const float* norm_w;                 // [rank]
    const float* freq; float rot_gain;   // [rot_dims / 2]; factor on cos and sin
    float eps;
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    void* cache; int num_slots;          // [num_slots, rank + rot_dim]
    void* q_rot;                         // [T, heads, rot_dim]
    int* guard;
};

constexpr int PRE_Q = 1024;              // rotated query values per block

// grid (T, 1 + ceil(heads * rot_dim / PRE_Q)), block 256: block y = 0 makes the cache row, the others rotate query parts
template <typename T>
__global__ void __launch_bounds__(256) latent_pre_kernel(LatentPreParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x, half = p.rot_dims / 2;
    float* cs = sm;
    float* sn = sm + half;
    const int pos = p.positions[t];
    const T* row = (const T*)p.qd + (size_t)t * p.ld;
    const int qs = p.dim + p.rot_dim;
    for (int i = tid; i < half; i += 256) {
        float a, b;
        sincosf((float)pos * p.freq[i], &a, &b);
        sn[i] = a * p.rot_gain;
        cs[i] = b * p.rot_gain;
    }
    // value i of a rotated part that starts at x
    auto rotated = [&](const T* x, int i) {
        const float v = to_f(x[i]);
        if (i < half) return v * cs[i] - to_f(x[i + half]) * sn[i];
        if (i < p.rot_dims) return v * cs[i - half] + to_f(x[i - half]) * sn[i - half];
        return v;
    };
    if (blockIdx.y > 0) {
        __syncthreads();
        T* qo = (T*)p.q_rot + (size_t)t * p.heads * p.rot_dim;
        const int j0 = (blockIdx.y - 1) * PRE_Q, total = p.heads * p.rot_dim;
#pragma unroll
        for (int u = 0; u < PRE_Q / 256; ++u) {
            const int j = j0 + u * 256 + tid;
            if (j < total) put(qo + j, rotated(row + (size_t)(j / p.rot_dim) * qs + p.dim, j % p.rot_dim));
        }
        return;
    }
    const int page = p.page_table[(size_t)p.batch_idx[t] * p.pt_stride + pos / p.page_size];
    const long long slot = (long long)page * p.page_size + pos % p.page_size;
    const T* lat = row + (size_t)p.heads * qs;
    float ss = 0.f;
#pragma unroll 4
    for (int i = tid; i < p.rank; i += 256) {
        const float v = to_f(lat[i]);
        ss += v * v;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)p.rank + p.eps);      // (also orders the cos / sin table)
    if (!guard_ok(p.guard, 21, slot, p.num_slots)) return;
    T* dst = (T*)p.cache + (size_t)slot * (p.rank + p.rot_dim);
#pragma unroll 4
    for (int i = tid; i < p.rank; i += 256) put(dst + i, to_f(lat[i]) * inv * p.norm_w[i]);
    for (int i = tid; i < p.rot_dim; i += 256) put(dst + p.rank + i, rotated(lat + p.rank, i));
}

struct LatentRowsParams {
    const void* q_abs;                   // [T, heads, rank]
    const void* q_rot;                   // [T, heads, rot_dim]
    const void* cache; int num_slots;
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    int heads, rank, rot_dim, window;    // window 0: every earlier position
    float scale;
    const float* sink;                   // [heads] or null
    void* out;                           // [T, heads, rank]
    int* guard;
};

constexpr int ROWS_KT = 64;              // keys per tile
constexpr int ROWS_MAXV = 8;             // latent values per thread (rank <= 128 * 8)

// grid (heads, T), block 128
template <typename T>
__global__ void __launch_bounds__(128) latent_rows_kernel(LatentRowsParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    __shared__ float sc[ROWS_KT];
    __shared__ long long slots[ROWS_KT];
    __shared__ float scratch[33];
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int D = p.rank + p.rot_dim;
    float* q = sm;
    for (int i = tid; i < p.rank; i += 128) q[i] = to_f(((const T*)p.q_abs)[((size_t)t * p.heads + h) * p.rank + i]);
    for (int i = tid; i < p.rot_dim; i += 128) q[p.rank + i] = to_f(((const T*)p.q_rot)[((size_t)t * p.heads + h) * p.rot_dim + i]);
    const int pos = p.positions[t];
    const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
    const int* pt = p.page_table + (size_t)p.batch_idx[t] * p.pt_stride;
    const T* cache = (const T*)p.cache;
    float m = p.sink != nullptr ? p.sink[h] : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f;
    float o[ROWS_MAXV];
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) o[i] = 0.f;
    for (int k0 = first; k0 <= pos; k0 += ROWS_KT) {
        const int nk = min(ROWS_KT, pos + 1 - k0);
        __syncthreads();
        if (tid < nk) {
            const int kp = k0 + tid;
            const long long s = (long long)pt[kp / p.page_size] * p.page_size + kp % p.page_size;
            slots[tid] = guard_ok(p.guard, 22, s, p.num_slots) ? s : 0;
        }
        __syncthreads();
        for (int k = warp; k < nk; k += 4) {
            const T* row = cache + (size_t)slots[k] * D;
            float a = 0.f;
            for (int i = lane; i < D; i += 32) a += q[i] * to_f(row[i]);
            a = warp_sum(a);
            if (lane == 0) sc[k] = a * p.scale;
        }
        __syncthreads();
        const float top = fmaxf(m, block_max(tid < nk ? sc[tid] : -FLT_MAX, scratch));
        const float e = tid < nk ? expf(sc[tid] - top) : 0.f;
        const float f = m == -INFINITY ? 0.f : expf(m - top);
        const float sum = block_sum(e, scratch);
        if (tid < nk) sc[tid] = e;
        l = l * f + sum;
        m = top;
        __syncthreads();
#pragma unroll
        for (int i = 0; i < ROWS_MAXV; ++i) {
            const int d = tid + i * 128;
            if (d >= p.rank) break;
            float a = o[i] * f;
            for (int k = 0; k < nk; ++k) a += sc[k] * to_f(cache[(size_t)slots[k] * D + d]);
            o[i] = a;
        }
    }
    const float inv = 1.f / l;
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) {
        const int d = tid + i * 128;
        if (d < p.rank) put((T*)p.out + ((size_t)t * p.heads + h) * p.rank + d, o[i] * inv);
    }
}

}  // namespace

SL_API int sl_latent_pre(const LatentPreParams* p, int T, int f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->rot_dims > p->rot_dim || p->rot_dims % 2 != 0) return -1;
    const size_t smem = (size_t)p->rot_dims * sizeof(float);
    const dim3 grid(T, 1 + (p->heads * p->rot_dim + PRE_Q - 1) / PRE_Q);
    if (f32) sl_launch(latent_pre_kernel<float>, grid, 256, smem, s, *p);
    else sl_launch(latent_pre_kernel<bf16>, grid, 256, smem, s, *p);
    return SL_LAUNCH_CHECK();
}

SL_API int sl_latent_rows(const LatentRowsParams* p, int T, int f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->rank > 128 * ROWS_MAXV || T > 65535) return -1;
    const size_t smem = (size_t)(p->rank + p->rot_dim) * sizeof(float);
    if (smem > 40 * 1024) return -1;
    if (f32) sl_launch(latent_rows_kernel<float>, dim3(p->heads, T), 128, smem, s, *p);
    else sl_launch(latent_rows_kernel<bf16>, dim3(p->heads, T), 128, smem, s, *p);
    return SL_LAUNCH_CHECK();
}
