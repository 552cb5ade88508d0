// Talking heads over a paged cache: grouped-query attention whose query heads' scores are mixed before the softmax,
//
//   s_h[j] = sum_g talk[h, g] * scale * q_g . k_j[key head of g],      o_h = softmax_j(s_h[j]) . v_j[value head of h],
//
// with positions that see their own chunk of the sequence only.
//
//  * talking_rows_kernel: independent token rows on the CUDA cores, any sizes, bf16 or fp32.
#include "common.cuh"
#include "mma_sync.cuh"

namespace {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

struct TalkingParams {
    const void* q;                       // [T, heads, dim]
    const void *k_cache, *v_cache; int num_slots;        // [slots, kv_heads, dim], [slots, v_heads, vdim]
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    int heads, kv_heads, out_heads, v_heads, dim, vdim, chunk;
    float scale;
    const float* talk;                   // [out_heads, heads]
    void* out; int ldo;                  // [T, ldo]: output head h at h * vdim
    int* guard;
};

constexpr int ROWS_KT = 32, ROWS_THREADS = 256;

__host__ __device__ inline size_t rows_smem_floats(int heads, int out_heads, int dim, int vdim) {
    return (size_t)heads * dim + (size_t)out_heads * vdim + (size_t)(heads + out_heads) * ROWS_KT + 3 * out_heads;
}

// grid T, block 256
template <typename T>
__global__ void __launch_bounds__(ROWS_THREADS) talking_rows_kernel(TalkingParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    __shared__ long long slots[ROWS_KT];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int nq = p.heads * p.dim, no = p.out_heads * p.vdim, kgroup = p.heads / p.kv_heads, vgroup = p.out_heads / p.v_heads;
    float *q = sm, *o = q + nq, *raw = o + no, *sc = raw + p.heads * ROWS_KT, *m = sc + p.out_heads * ROWS_KT, *l = m + p.out_heads, *f = l + p.out_heads;
    const int pos = p.positions[t], lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
    const int* pt = p.page_table + (size_t)p.batch_idx[t] * p.pt_stride;
    for (int i = tid; i < nq; i += ROWS_THREADS) q[i] = to_f(((const T*)p.q)[(size_t)t * nq + i]) * p.scale;
    for (int i = tid; i < no; i += ROWS_THREADS) o[i] = 0.f;
    for (int i = tid; i < p.out_heads; i += ROWS_THREADS) { m[i] = -INFINITY; l[i] = 0.f; }
    const size_t krow = (size_t)p.kv_heads * p.dim, vrow = (size_t)p.v_heads * p.vdim;
    for (int k0 = lo; k0 <= pos; k0 += ROWS_KT) {
        const int nk = min(ROWS_KT, pos + 1 - k0);
        __syncthreads();
        if (tid < nk) {
            const int kp = k0 + tid;
            const long long s = (long long)pt[kp / p.page_size] * p.page_size + kp % p.page_size;
            slots[tid] = guard_ok(p.guard, 31, s, p.num_slots) ? s : 0;
        }
        __syncthreads();
        // a warp takes a key head of a key: its values serve the whole group of query heads
        for (int u = warp; u < nk * p.kv_heads; u += ROWS_THREADS / 32) {
            const int k = u / p.kv_heads, hk = u - k * p.kv_heads;
            const T* row = (const T*)p.k_cache + (size_t)slots[k] * krow + (size_t)hk * p.dim;
            for (int g = hk * kgroup; g < (hk + 1) * kgroup; ++g) {
                float a = 0.f;
                for (int i = lane; i < p.dim; i += 32) a += q[g * p.dim + i] * to_f(row[i]);
                a = warp_sum(a);
                if (lane == 0) raw[g * ROWS_KT + k] = a;
            }
        }
        __syncthreads();
        for (int u = tid; u < p.out_heads * ROWS_KT; u += ROWS_THREADS) {
            const int h = u / ROWS_KT, k = u % ROWS_KT;
            float a = 0.f;
            for (int g = 0; g < p.heads && k < nk; ++g) a += p.talk[h * p.heads + g] * raw[g * ROWS_KT + k];
            sc[u] = k < nk ? a : -INFINITY;
        }
        __syncthreads();
        for (int h = warp; h < p.out_heads; h += ROWS_THREADS / 32) {
            const float s = sc[h * ROWS_KT + lane], top = fmaxf(m[h], warp_max(s)), e = expf(s - top);
            const float sum = warp_sum(e), factor = expf(m[h] - top);
            __syncwarp();
            sc[h * ROWS_KT + lane] = e;
            if (lane == 0) {
                f[h] = factor;
                l[h] = l[h] * factor + sum;
                m[h] = top;
            }
        }
        __syncthreads();
        for (int i = tid; i < no; i += ROWS_THREADS) {
            const int h = i / p.vdim, d = i - h * p.vdim;
            const T* v = (const T*)p.v_cache + (size_t)(h / vgroup) * p.vdim + d;
            float a = o[i] * f[h];
            for (int k = 0; k < nk; ++k) a += sc[h * ROWS_KT + k] * to_f(v[(size_t)slots[k] * vrow]);
            o[i] = a;
        }
    }
    __syncthreads();
    for (int i = tid; i < no; i += ROWS_THREADS) put((T*)p.out + (size_t)t * p.ldo + i, o[i] / l[i / p.vdim]);
}

bool shape_ok(const TalkingParams* p) {
    return p->heads >= 1 && p->kv_heads >= 1 && p->out_heads >= 1 && p->v_heads >= 1 && p->heads % p->kv_heads == 0 && p->out_heads % p->v_heads == 0 &&
           p->chunk >= 0;
}

}  // namespace

SL_API int sl_talking_rows(const TalkingParams* p, int T, int f32, cudaStream_t s) {
    if (T == 0) return 0;
    const size_t smem = rows_smem_floats(p->heads, p->out_heads, p->dim, p->vdim) * sizeof(float);
    if (!shape_ok(p) || smem > 200 * 1024) return -1;
    auto go = [&](auto kern) {
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        sl_launch(kern, T, ROWS_THREADS, smem, s, *p);
        return SL_LAUNCH_CHECK();
    };
    return f32 ? go(talking_rows_kernel<float>) : go(talking_rows_kernel<bf16>);
}
