// Residual stream of decoders that normalise a sublayer's output before it is added ("sandwich" norms):
//
//   residual' = residual + rms(y) * w_post          (y: the sublayer's output, fp32; absent in front of the first sublayer)
//   out       = rms(residual') * w_next             (input of the next sublayer, or of the output head)
//
// in one pass over the token's row, which stays in registers between the two reductions.  The first call of a step gathers
// the residual from the embedding table instead.  Weights, sums and the residual are fp32; `out` is bf16 or fp32.
#include "common.cuh"

namespace {

struct PostNormParams {
    void* out; int out_f32;          // [T, H]
    float* res_out;                  // [T, H]
    const float* y; int ldy;         // [T, ldy] or null
    const float* w_post;             // [H] (with y)
    const float* res_in;             // [T, H] or null: gathered from `table`
    const long long* ids; const void* table; int table_f32, vocab;
    const float* w_next;             // [H]
    int H; float eps;
};

// one block per token, thread holds values tid, tid + blockDim, ...
template <int NV>
__global__ void __launch_bounds__(1024) post_norm_kernel(PostNormParams p) {
    pdl_grid_sync();
    __shared__ float scratch[33];
    const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x, H = p.H;
    float r[NV];
    if (p.res_in != nullptr) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = tid + i * nt;
            r[i] = c < H ? p.res_in[(size_t)t * H + c] : 0.f;
        }
    } else {
        long long id = p.ids[t];
        id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);      // never read outside the table
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = tid + i * nt;
            r[i] = c >= H ? 0.f : p.table_f32 ? ((const float*)p.table)[(size_t)id * H + c]
                                              : __bfloat162float(((const bf16*)p.table)[(size_t)id * H + c]);
        }
    }
    if (p.y != nullptr) {
        float y[NV], ss = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = tid + i * nt;
            y[i] = c < H ? p.y[(size_t)t * p.ldy + c] : 0.f;
            ss += y[i] * y[i];
        }
        const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + p.eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = tid + i * nt;
            if (c < H) r[i] += y[i] * inv * p.w_post[c];
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) ss += r[i] * r[i];
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)H + p.eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = tid + i * nt;
        if (c >= H) continue;
        p.res_out[(size_t)t * H + c] = r[i];
        const float o = r[i] * inv * p.w_next[c];
        if (p.out_f32) ((float*)p.out)[(size_t)t * H + c] = o;
        else ((bf16*)p.out)[(size_t)t * H + c] = __float2bfloat16(o);
    }
}

}  // namespace

SL_API int sl_post_norm(const PostNormParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->H < 1 || p->H > 16384 || (p->res_in == nullptr && p->table == nullptr)) return -1;
    int nt = (p->H / 4 + 31) / 32 * 32;
    nt = nt < 64 ? 64 : (nt > 1024 ? 1024 : nt);
    const int per = (p->H + nt - 1) / nt;
    if (per <= 4) sl_launch(post_norm_kernel<4>, T, nt, 0, s, *p);
    else if (per <= 8) sl_launch(post_norm_kernel<8>, T, nt, 0, s, *p);
    else sl_launch(post_norm_kernel<16>, T, nt, 0, s, *p);
    return SL_LAUNCH_CHECK();
}
