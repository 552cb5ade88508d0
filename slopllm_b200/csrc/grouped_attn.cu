// Grouped-query attention over a paged cache: query / key norm, rotary table, sliding window with kept first tokens, softmax
// sink, values of their own or the key projections themselves.  (Portions of prompts attend in latent_mma.cu.)
//
//  * grouped_pre_kernel: biases, per-head RMS norm and rotate-half of queries and keys; keys and values go into their cache slots.
//  * grouped_row_pre_kernel: the same step for norms over the whole query / key rows: biases, norms, rotation of adjacent pairs from
//    a table of angles, a factor per query head, and values that turn with their position.
//  * grouped_rows_kernel: independent token rows on the CUDA cores, any sizes, bf16 or fp32.
//  * grouped_decode_kernel: one query token per page-table row on the tensor cores: a CTA takes the query heads of one key head
//    (16 at a time) x a range of the visible keys, which come through two cp.async stages.  grouped_merge_kernel joins the key
//    splits; the sink belongs to split 0, so it counts once.
//
// Values that were turned by their position are turned back by the query's when a row's sum is complete (`turn`): every kernel
// holds the adjacent values of a pair in one thread (or two neighbouring lanes) then.
//
// The keys that a row sees are numbered 0 .. n-1: first the kept ones before the window, then the window.
#include "common.cuh"
#include "mma_sync.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }

struct GroupedPreParams {
    const void *q, *k, *v; int ld;       // token-major projection rows (v may be k)
    int heads, kv_heads, dim, vdim, rot_dims;
    const float *q_norm, *k_norm;        // [dim] or null
    const float* freq; float rot_gain, eps;
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    void *k_cache, *v_cache; int num_slots;      // [slots, kv_heads, dim], [slots, v_heads, vdim]
    void* q_out;                         // [T, heads, dim]
    int* guard;
    int v_heads;                         // at most kv_heads
    const float *q_bias, *k_bias, *v_bias;       // per projection row, or null
};

// grid (T, ceil((heads + kv_heads) / 8)), block 256: a warp per head
template <typename TI, typename TO>
__global__ void __launch_bounds__(256) grouped_pre_kernel(GroupedPreParams p) {
    pdl_grid_sync();
    extern __shared__ float sm[];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, half = p.rot_dims / 2;
    float *cs = sm, *sn = cs + half, *x = sn + half + warp * p.dim;
    const int pos = p.positions[t];
    for (int i = tid; i < half; i += 256) {
        float a, b;
        sincosf((float)pos * p.freq[i], &a, &b);
        sn[i] = a * p.rot_gain;
        cs[i] = b * p.rot_gain;
    }
    const int hh = blockIdx.y * 8 + warp;
    const bool is_q = hh < p.heads, on = hh < p.heads + p.kv_heads;
    const int h = is_q ? hh : hh - p.heads;
    const float* w = is_q ? p.q_norm : p.k_norm;
    float inv = 1.f;
    if (on) {
        const TI* src = (const TI*)(is_q ? p.q : p.k) + (size_t)t * p.ld + (size_t)h * p.dim;
        const float* bias = is_q ? p.q_bias : p.k_bias;
        float ss = 0.f;
        for (int i = lane; i < p.dim; i += 32) {
            const float v = to_f(src[i]) + (bias != nullptr ? bias[h * p.dim + i] : 0.f);
            x[i] = v;
            ss += v * v;
        }
        if (w != nullptr) inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
        __syncwarp();
        if (w != nullptr)
            for (int i = lane; i < p.dim; i += 32) x[i] = x[i] * inv * w[i];
    }
    __syncthreads();
    if (!on) return;
    TO* dst;
    if (is_q) {
        dst = (TO*)p.q_out + ((size_t)t * p.heads + h) * p.dim;
    } else {
        const int page = p.page_table[(size_t)p.batch_idx[t] * p.pt_stride + pos / p.page_size];
        const long long slot = (long long)page * p.page_size + pos % p.page_size;
        if (!guard_ok(p.guard, 25, slot, p.num_slots)) return;
        dst = (TO*)p.k_cache + ((size_t)slot * p.kv_heads + h) * p.dim;
        const TI* vs = (const TI*)p.v + (size_t)t * p.ld + (size_t)h * p.vdim;
        TO* vd = (TO*)p.v_cache + ((size_t)slot * p.v_heads + h) * p.vdim;
        if (h < p.v_heads)
            for (int i = lane; i < p.vdim; i += 32) put(vd + i, to_f(vs[i]) + (p.v_bias != nullptr ? p.v_bias[h * p.vdim + i] : 0.f));
    }
    for (int i = lane; i < p.dim; i += 32) {
        float v = x[i];
        if (i < half) v = v * cs[i] - x[i + half] * sn[i];
        else if (i < p.rot_dims) v = v * cs[i - half] + x[i - half] * sn[i - half];
        put(dst + i, v);
    }
}

struct GroupedRowPreParams {
    const void *q, *k, *v; int ld;       // token-major projection rows
    int heads, kv_heads, dim, vdim, rot_dims;
    const float *q_bias, *k_bias, *v_bias;       // per projection row, or null
    const float *q_norm, *k_norm;        // [heads * dim], [kv_heads * dim]
    const float* sums;                   // [T, 2] sums of squares of the whole rows, or null: this launch's own rows are whole
    float q_count, k_count, eps;         // values of a whole row
    const float* gain;                   // [heads] factor on a head's queries, or null
    const float2 *qk_turn, *v_turn; int ldt;     // (cos, sin) of pair m of token t at t * ldt + m (v_turn null: values do not turn)
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    void *k_cache, *v_cache; int num_slots;      // [slots, kv_heads, dim], [slots, kv_heads, vdim]
    void* q_out;                         // [T, heads, dim]
    int* guard;
};

__device__ __forceinline__ float2 turned(float2 x, float2 cs) { return make_float2(x.x * cs.x - x.y * cs.y, x.y * cs.x + x.x * cs.y); }
__device__ __forceinline__ float2 turned_back(float2 x, float2 cs) { return make_float2(x.x * cs.x + x.y * cs.y, x.y * cs.x - x.x * cs.y); }

// VW consecutive values: 1, 2, or 8 (16-byte accesses)
template <int VW>
struct Piece { float v[VW]; };
template <int VW>
__device__ __forceinline__ Piece<VW> load_piece(const float* p) {
    Piece<VW> x;
    if (VW == 1) x.v[0] = *p;
    else if (VW == 2) *reinterpret_cast<float2*>(x.v) = *reinterpret_cast<const float2*>(p);
    else
#pragma unroll
        for (int i = 0; i < VW; i += 4) *reinterpret_cast<float4*>(x.v + i) = *reinterpret_cast<const float4*>(p + i);
    return x;
}
template <int VW>
__device__ __forceinline__ Piece<VW> load_piece(const bf16* p) {
    Piece<VW> x;
    if (VW == 1) {
        x.v[0] = to_f(*p);
    } else {
        uint32_t w[VW / 2 + 1];
        if (VW == 8) *reinterpret_cast<uint4*>(w) = *reinterpret_cast<const uint4*>(p);
        else w[0] = *reinterpret_cast<const uint32_t*>(p);
#pragma unroll
        for (int i = 0; i + 1 < VW; i += 2) *reinterpret_cast<float2*>(x.v + i) = bf162_to_f2(w[i / 2]);
    }
    return x;
}
template <int VW>
__device__ __forceinline__ void store_piece(float* p, const Piece<VW>& x) {
    if (VW == 1) *p = x.v[0];
    else if (VW == 2) *reinterpret_cast<float2*>(p) = *reinterpret_cast<const float2*>(x.v);
    else
#pragma unroll
        for (int i = 0; i < VW; i += 4) *reinterpret_cast<float4*>(p + i) = *reinterpret_cast<const float4*>(x.v + i);
}
template <int VW>
__device__ __forceinline__ void store_piece(bf16* p, const Piece<VW>& x) {
    if (VW == 1) {
        put(p, x.v[0]);
    } else {
        uint32_t w[VW / 2 + 1];
#pragma unroll
        for (int i = 0; i + 1 < VW; i += 2) w[i / 2] = f2_to_bf162(x.v[i], x.v[i + 1]);
        if (VW == 8) *reinterpret_cast<uint4*>(p) = *reinterpret_cast<const uint4*>(w);
        else *reinterpret_cast<uint32_t*>(p) = w[0];
    }
}
template <int VW>
__device__ __forceinline__ void add_piece(Piece<VW>& x, const float* b) {
    if (b == nullptr) return;
    const Piece<VW> y = load_piece<VW>(b);
#pragma unroll
    for (int i = 0; i < VW; ++i) x.v[i] += y.v[i];
}

// A block per token, a thread takes pieces of VW values (of one head); with single values it looks up their partners.
template <int VW, typename TI, typename TO>
__global__ void __launch_bounds__(1024) grouped_row_pre_kernel(GroupedRowPreParams p) {
    pdl_grid_sync();
    extern __shared__ __align__(16) float row[];         // [heads * dim | kv_heads * dim] with biases
    __shared__ float part[2][32];
    const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, step = blockDim.x * VW;
    const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim, nv = p.kv_heads * p.vdim, pos = p.positions[t];
    const TI *q = (const TI*)p.q + (size_t)t * p.ld, *k = (const TI*)p.k + (size_t)t * p.ld, *v = (const TI*)p.v + (size_t)t * p.ld;
    const int page = p.page_table[(size_t)p.batch_idx[t] * p.pt_stride + pos / p.page_size];
    // a row with its biases -> shared, and the sum of its squares
    auto read = [&](const TI* src, const float* bias, float* dst, int n) {
        float ss = 0.f;
#pragma unroll 2
        for (int i = tid * VW; i < n; i += step) {
            Piece<VW> x = load_piece<VW>(src + i);
            add_piece<VW>(x, bias != nullptr ? bias + i : nullptr);
            store_piece<VW>(dst + i, x);
#pragma unroll
            for (int j = 0; j < VW; ++j) ss += x.v[j] * x.v[j];
        }
        return warp_sum(ss);
    };
    float sq = read(q, p.q_bias, row, nq), sk = read(k, p.k_bias, row + nq, nk);
    if (lane == 0) { part[0][warp] = sq; part[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.f;
    for (int i = 0; i < blockDim.x >> 5; ++i) { sq += part[0][i]; sk += part[1][i]; }
    if (p.sums != nullptr) { sq = p.sums[t * 2]; sk = p.sums[t * 2 + 1]; }
    const float iq = 1.f / sqrtf(sq / p.q_count + p.eps), ik = 1.f / sqrtf(sk / p.k_count + p.eps);
    // pieces of a head at place d; the partner of a single value is `partner`
    auto turn_piece = [&](Piece<VW>& x, const float2* turn, int d, int dims, float partner) {
        if (VW == 1) {
            if (d < dims) {
                const float2 cs = turn[d >> 1];
                x.v[0] = x.v[0] * cs.x + (d & 1 ? partner : -partner) * cs.y;
            }
            return;
        }
#pragma unroll
        for (int j = 0; j + 1 < VW; j += 2) {
            if (d + j >= dims) break;
            const float2 y = turned(make_float2(x.v[j], x.v[j + 1]), turn[(d + j) >> 1]);
            x.v[j] = y.x;
            x.v[j + 1] = y.y;
        }
    };
    const float2* qk_turn = p.qk_turn + (size_t)t * p.ldt;
    auto finish = [&](const float* src, const float* w, float inv, const float* gain, TO* dst, int n) {
#pragma unroll 2
        for (int i = tid * VW; i < n; i += step) {
            const int h = i / p.dim, d = i - h * p.dim;
            const float f = gain != nullptr ? inv * gain[h] : inv;
            Piece<VW> x = load_piece<VW>(src + i);
            const Piece<VW> g = load_piece<VW>(w + i);
#pragma unroll
            for (int j = 0; j < VW; ++j) x.v[j] *= f * g.v[j];
            const int o = i + (d & 1 ? -1 : 1);
            turn_piece(x, qk_turn, d, p.rot_dims, VW == 1 && d < p.rot_dims ? src[o] * f * w[o] : 0.f);
            store_piece<VW>(dst + i, x);
        }
    };
    finish(row, p.q_norm, iq, p.gain, (TO*)p.q_out + (size_t)t * nq, nq);
    const long long slot = (long long)page * p.page_size + pos % p.page_size;
    if (!guard_ok(p.guard, 28, slot, p.num_slots)) return;
    finish(row + nq, p.k_norm, ik, nullptr, (TO*)p.k_cache + (size_t)slot * nk, nk);
    TO* vd = (TO*)p.v_cache + (size_t)slot * nv;
    for (int i = tid * VW; i < nv; i += step) {
        Piece<VW> x = load_piece<VW>(v + i);
        add_piece<VW>(x, p.v_bias != nullptr ? p.v_bias + i : nullptr);
        if (p.v_turn != nullptr) {
            const int d = i % p.vdim, o = i + (d & 1 ? -1 : 1);
            turn_piece(x, p.v_turn + (size_t)t * p.ldt, d, p.vdim, VW == 1 ? to_f(v[o]) + (p.v_bias != nullptr ? p.v_bias[o] : 0.f) : 0.f);
        }
        store_piece<VW>(vd + i, x);
    }
}

// out[t] = sums of squares of the query and key rows with their biases: what a rank that holds some of the heads adds to the norms.
// grid T, block 256
template <typename TI>
__global__ void __launch_bounds__(256) row_sums_kernel(float* __restrict__ out, GroupedRowPreParams p) {
    pdl_grid_sync();
    __shared__ float scratch[33];
    const int t = blockIdx.x, nq = p.heads * p.dim, nk = p.kv_heads * p.dim;
    const TI *q = (const TI*)p.q + (size_t)t * p.ld, *k = (const TI*)p.k + (size_t)t * p.ld;
    float sq = 0.f, sk = 0.f;
    for (int i = threadIdx.x; i < nq + nk; i += 256) {
        const bool is_q = i < nq;
        const int j = is_q ? i : i - nq;
        const float* b = is_q ? p.q_bias : p.k_bias;
        const float x = to_f(is_q ? q[j] : k[j]) + (b != nullptr ? b[j] : 0.f);
        (is_q ? sq : sk) += x * x;
    }
    sq = block_sum(sq, scratch);
    sk = block_sum(sk, scratch);
    if (threadIdx.x == 0) { out[t * 2] = sq; out[t * 2 + 1] = sk; }
}

struct GroupedAttnParams {
    const void* q;                       // [T, heads, dim]
    const void *k_cache, *v_cache; int num_slots;
    const int* positions; const int* batch_idx; const int* page_table;
    int pt_stride, page_size;
    int heads, kv_heads, dim, vdim, window, keep_first, splits;
    float scale;
    const float* sink;                   // [heads] or null
    void* out; int ldo;                  // [T, ldo]: head h at h * vdim
    float *o_part, *lse_part;            // [T, heads, splits, vdim], [T, heads, splits] (decode with more than one split)
    int* guard;
    const float2* turn; int ldt;         // (cos, sin) by which pair m of token t's values is turned back, at t * ldt + m (or null)
    float out_scale;                     // factor on the output
};

__device__ __forceinline__ float2 finished(const GroupedAttnParams& p, int t, int d, float x, float y) {
    return p.turn == nullptr ? make_float2(x, y) : turned_back(make_float2(x, y), p.turn[(size_t)t * p.ldt + (d >> 1)]);
}

// The keys a position sees: n of them, number i is position at(i).
struct Visible {
    int kept, first, n;
    __device__ __forceinline__ Visible(const GroupedAttnParams& p, int pos) {
        first = p.window > 0 ? max(0, pos - p.window + 1) : 0;
        kept = min(p.keep_first, first);
        n = kept + pos + 1 - first;
    }
    __device__ __forceinline__ int at(int i) const { return i < kept ? i : first + i - kept; }
};

constexpr int ROWS_KT = 64, ROWS_MAXV = 4;      // keys per tile; values per thread (vdim <= 512)

// grid (heads, T), block 128
template <typename T>
__global__ void __launch_bounds__(128) grouped_rows_kernel(GroupedAttnParams p) {
    pdl_grid_sync();
    extern __shared__ float q[];
    __shared__ float sc[ROWS_KT];
    __shared__ long long slots[ROWS_KT];
    __shared__ float scratch[33];
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int hkv = h / (p.heads / p.kv_heads);
    for (int i = tid; i < p.dim; i += 128) q[i] = to_f(((const T*)p.q)[((size_t)t * p.heads + h) * p.dim + i]);
    const Visible vis(p, p.positions[t]);
    const int* pt = p.page_table + (size_t)p.batch_idx[t] * p.pt_stride;
    const T *kc = (const T*)p.k_cache + (size_t)hkv * p.dim, *vc = (const T*)p.v_cache + (size_t)hkv * p.vdim;
    const size_t krow = (size_t)p.kv_heads * p.dim, vrow = (size_t)p.kv_heads * p.vdim;
    float m = p.sink != nullptr ? p.sink[h] : -INFINITY, l = p.sink != nullptr ? 1.f : 0.f;
    float o[ROWS_MAXV];
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) o[i] = 0.f;
    for (int k0 = 0; k0 < vis.n; k0 += ROWS_KT) {
        const int nk = min(ROWS_KT, vis.n - k0);
        __syncthreads();
        if (tid < nk) {
            const int kp = vis.at(k0 + tid);
            const long long s = (long long)pt[kp / p.page_size] * p.page_size + kp % p.page_size;
            slots[tid] = guard_ok(p.guard, 26, s, p.num_slots) ? s : 0;
        }
        __syncthreads();
        for (int k = warp; k < nk; k += 4) {
            const T* row = kc + (size_t)slots[k] * krow;
            float a = 0.f;
            for (int i = lane; i < p.dim; i += 32) a += q[i] * to_f(row[i]);
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
            if (d >= p.vdim) break;
            float a = o[i] * f;
            for (int k = 0; k < nk; ++k) a += sc[k] * to_f(vc[(size_t)slots[k] * vrow + d]);
            o[i] = a;
        }
    }
    const float inv = p.out_scale / l;
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) {
        const int d = tid + i * 128;
        const float x = o[i] * inv, y = __shfl_xor_sync(0xffffffffu, x, 1);
        if (d >= p.vdim) continue;
        const float2 f = d & 1 ? finished(p, t, d, y, x) : finished(p, t, d, x, y);
        put((T*)p.out + (size_t)t * p.ldo + (size_t)h * p.vdim + d, d & 1 ? f.y : f.x);
    }
}

constexpr int KT = 64, STAGES = 2, DT = 128;     // keys per tile, threads of the decode kernel

// grid (splits, kv_heads * head groups of 16, T), block 128.  NTW: 8-wide value tiles per warp (vdim <= 32 * NTW).
template <int NTW>
__global__ void __launch_bounds__(DT) grouped_decode_kernel(GroupedAttnParams p) {
    pdl_grid_sync();
    extern __shared__ __align__(16) unsigned char smraw[];
    const int group = p.heads / p.kv_heads, hg = (group + 15) / 16;
    const int split = blockIdx.x, hkv = blockIdx.y / hg, t = blockIdx.z;
    const int r_lo = blockIdx.y % hg * 16, nr = min(16, group - r_lo), h0 = hkv * group + r_lo;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, c4 = lane & 3;
    const int dqp = (p.dim + 15) / 16 * 16, ld = dqp + 8, ldv = p.vdim + 8;
    bf16* qs = reinterpret_cast<bf16*>(smraw);                      // [16][ld]
    bf16* ks = qs + 16 * ld;                                        // STAGES x [KT][ld]
    bf16* vs = ks + STAGES * KT * ld;                               // STAGES x [KT][ldv]
    float* sc = reinterpret_cast<float*>(vs + STAGES * KT * ldv);   // [16][KT + 4]
    bf16* ph = reinterpret_cast<bf16*>(sc + 16 * (KT + 4));         // [16][KT + 8]
    bf16* pl = ph + 16 * (KT + 8);
    float* fac = reinterpret_cast<float*>(pl + 16 * (KT + 8));      // [16]
    const Visible vis(p, p.positions[t]);
    const int tiles = (vis.n + KT - 1) / KT, per = (tiles + p.splits - 1) / p.splits;
    const int tb = min(tiles, split * per), te = min(tiles, tb + per);
    const int* pt = p.page_table + (size_t)p.batch_idx[t] * p.pt_stride;
    const bf16 *kc = (const bf16*)p.k_cache + (size_t)hkv * p.dim, *vc = (const bf16*)p.v_cache + (size_t)hkv * p.vdim;
    const size_t krow = (size_t)p.kv_heads * p.dim, vrow = (size_t)p.kv_heads * p.vdim;
    const int kpc = p.dim / 8, vpc = p.vdim / 8;
    // a warp fetches 16 rows of a tile
    auto fetch = [&](int j) {
        if (j < te) {
            const int k0 = j * KT, nk = min(KT, vis.n - k0), st = (j - tb) % STAGES;
            long long slot = -1;
            if (lane < 16 && warp * 16 + lane < nk) {
                const int kp = vis.at(k0 + warp * 16 + lane);
                const long long s = (long long)pt[kp / p.page_size] * p.page_size + kp % p.page_size;
                slot = guard_ok(p.guard, 27, s, p.num_slots) ? s : -1;
            }
            bf16 *kd = ks + (st * KT + warp * 16) * ld, *vd = vs + (st * KT + warp * 16) * ldv;
            // (all lanes take part in every shuffle: a lane that left its last round early could not be read)
            auto copy = [&](bf16* dst, int dld, const bf16* src, size_t row, int pieces) {
                int r = lane / pieces, c = lane - r * pieces;
                const int dr = 32 / pieces, dc = 32 - dr * pieces;
#pragma unroll 4
                for (int i0 = 0; i0 < 16 * pieces; i0 += 32) {
                    const long long s = __shfl_sync(0xffffffffu, slot, r & 15);
                    bf16* to = dst + r * dld + c * 8;
                    if (r < 16) {
                        if (s >= 0) cp_async16(to, src + (size_t)s * row + c * 8);
                        else *reinterpret_cast<uint4*>(to) = make_uint4(0, 0, 0, 0);
                    }
                    r += dr;
                    c += dc;
                    if (c >= pieces) { c -= pieces; ++r; }
                }
            };
            copy(kd, ld, kc, krow, kpc);
            copy(vd, ldv, vc, vrow, vpc);
        }
        cp_async_commit();
    };
    for (int i = tid; i < 16 * (dqp / 8); i += DT) {
        const int r = i / (dqp / 8), c = i % (dqp / 8) * 8;
        uint4 x = make_uint4(0, 0, 0, 0);
        if (r < nr && c < p.dim) x = *reinterpret_cast<const uint4*>((const bf16*)p.q + ((size_t)t * p.heads + h0 + r) * p.dim + c);
        *reinterpret_cast<uint4*>(qs + r * ld + c) = x;
    }
    if (dqp > p.dim)                                                // (dim % 8 == 0: one column piece of padding)
        for (int r = tid; r < STAGES * KT; r += DT) *reinterpret_cast<uint4*>(ks + r * ld + p.dim) = make_uint4(0, 0, 0, 0);
    float m[4], l[4];                                               // softmax state of rows 4 * warp ..
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int r = warp * 4 + u;
        const bool s = split == 0 && p.sink != nullptr && r < nr;
        m[u] = s ? p.sink[h0 + r] * LOG2E : -INFINITY;
        l[u] = s ? 1.f : 0.f;
    }
    const int nt = p.vdim / 8, tw = (nt + 3) / 4, n0 = warp * tw, nn = max(0, min(tw, nt - n0));
    float acc[NTW][4];
#pragma unroll
    for (int i = 0; i < NTW; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const float scale_log2 = p.scale * LOG2E;
    fetch(tb);
    for (int j = tb; j < te; ++j) {
        fetch(j + 1);
        cp_async_wait<1>();
        __syncthreads();
        const int nk = min(KT, vis.n - j * KT), st = (j - tb) % STAGES;
        const bf16 *kt = ks + st * KT * ld, *vt = vs + st * KT * ldv;
        float s4[2][4] = {};                                        // 16 heads x the warp's 16 keys
        for (int kk = 0; kk < dqp; kk += 16) {
            uint32_t a[4], b[4];
            ldsm_x4(a, qs + (lane & 15) * ld + kk + (lane >> 4) * 8);
            ldsm_x4(b, kt + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * ld + kk + ((lane >> 3) & 1) * 8);
            mma_bf16_16816(s4[0], a, b[0], b[1]);
            mma_bf16_16816(s4[1], a, b[2], b[3]);
        }
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int kcol = warp * 16 + u * 8 + c4 * 2;
            sc[g * (KT + 4) + kcol] = kcol < nk ? s4[u][0] * scale_log2 : -INFINITY;
            sc[g * (KT + 4) + kcol + 1] = kcol + 1 < nk ? s4[u][1] * scale_log2 : -INFINITY;
            sc[(g + 8) * (KT + 4) + kcol] = kcol < nk ? s4[u][2] * scale_log2 : -INFINITY;
            sc[(g + 8) * (KT + 4) + kcol + 1] = kcol + 1 < nk ? s4[u][3] * scale_log2 : -INFINITY;
        }
        __syncthreads();
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int r = warp * 4 + u;
            const float2 v = *reinterpret_cast<const float2*>(sc + r * (KT + 4) + lane * 2);
            const float x = fmaxf(m[u], warp_max(fmaxf(v.x, v.y)));
            const float f = m[u] == -INFINITY ? 0.f : exp2f(m[u] - x);
            const float e0 = exp2f(v.x - x), e1 = exp2f(v.y - x);
            l[u] = l[u] * f + warp_sum(e0 + e1);
            m[u] = x;
            uint32_t hi, lo;
            split_bf162(e0, e1, hi, lo);
            *reinterpret_cast<uint32_t*>(ph + r * (KT + 8) + lane * 2) = hi;
            *reinterpret_cast<uint32_t*>(pl + r * (KT + 8) + lane * 2) = lo;
            if (lane == 0) fac[r] = f;
        }
        __syncthreads();
        const float f0 = fac[g], f1 = fac[g + 8];
#pragma unroll
        for (int i = 0; i < NTW; ++i) { acc[i][0] *= f0; acc[i][1] *= f0; acc[i][2] *= f1; acc[i][3] *= f1; }
#pragma unroll
        for (int kk = 0; kk < KT; kk += 16) {
            uint32_t a[4], a2[4];
            ldsm_x4(a, ph + (lane & 15) * (KT + 8) + kk + (lane >> 4) * 8);
            ldsm_x4(a2, pl + (lane & 15) * (KT + 8) + kk + (lane >> 4) * 8);
#pragma unroll
            for (int i = 0; i < NTW; ++i) {
                if (i >= nn) break;
                uint32_t b0, b1;
                ldsm_x2_trans(b0, b1, vt + (kk + (lane & 15)) * ldv + (n0 + i) * 8);
                mma_bf16_16816(acc[i], a, b0, b1);
                mma_bf16_16816(acc[i], a2, b0, b1);
            }
        }
        __syncthreads();                                            // (the stage is filled again by the next fetch)
    }
    cp_async_wait_all();
#pragma unroll
    for (int u = 0; u < 4; ++u) {
        const int r = warp * 4 + u;
        if (lane == 0) {
            fac[r] = l[u] > 0.f ? (p.splits == 1 ? p.out_scale : 1.f) / l[u] : 0.f;
            if (r < nr && p.splits > 1)
                p.lse_part[((size_t)t * p.heads + h0 + r) * p.splits + split] = l[u] > 0.f ? (m[u] + log2f(l[u])) / LOG2E : -INFINITY;
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
            const int r = g + u * 8;
            if (r >= nr) continue;
            const float inv = u ? i1 : i0, x = acc[i][u * 2] * inv, y = acc[i][u * 2 + 1] * inv;
            if (p.splits == 1) {
                const float2 f = finished(p, t, d, x, y);
                *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)t * p.ldo + (size_t)(h0 + r) * p.vdim + d) = f2_to_bf162(f.x, f.y);
            } else *reinterpret_cast<float2*>(p.o_part + (((size_t)t * p.heads + h0 + r) * p.splits + split) * p.vdim + d) = make_float2(x, y);
        }
    }
}

// grid (heads, T), block 64: two values per thread and pass
__global__ void __launch_bounds__(64) grouped_merge_kernel(GroupedAttnParams p) {
    pdl_grid_sync();
    __shared__ float w[64];
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const size_t row = (size_t)t * p.heads + h;
    const float a = lane < p.splits ? p.lse_part[row * p.splits + lane] : -INFINITY;
    const float b = lane + 32 < p.splits ? p.lse_part[row * p.splits + lane + 32] : -INFINITY;
    const float top = warp_max(fmaxf(a, b));
    const float ea = a == -INFINITY ? 0.f : expf(a - top), eb = b == -INFINITY ? 0.f : expf(b - top);
    const float den = warp_sum(ea + eb), inv = den > 0.f ? p.out_scale / den : 0.f;
    if (tid < 32) {
        w[lane] = ea * inv;
        w[lane + 32] = eb * inv;
    }
    __syncthreads();
    for (int d = tid * 2; d < p.vdim; d += 128) {
        float x = 0.f, y = 0.f;
#pragma unroll 8
        for (int i = 0; i < p.splits; ++i) {
            const float2 v = *reinterpret_cast<const float2*>(p.o_part + (row * p.splits + i) * p.vdim + d);
            x += w[i] * v.x;
            y += w[i] * v.y;
        }
        const float2 f = finished(p, t, d, x, y);
        *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)t * p.ldo + (size_t)h * p.vdim + d) = f2_to_bf162(f.x, f.y);
    }
}

size_t decode_smem(int dim, int vdim) {
    const int ld = (dim + 15) / 16 * 16 + 8;
    return (size_t)16 * ld * 2 + (size_t)STAGES * KT * (ld + vdim + 8) * 2 + (size_t)16 * (KT + 4) * 4 + (size_t)2 * 16 * (KT + 8) * 2 + 64;
}

}  // namespace

SL_API int sl_grouped_pre(const GroupedPreParams* p, int T, int in_f32, int out_f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->rot_dims > p->dim || p->rot_dims % 2 != 0 || (out_f32 && !in_f32) || p->v_heads > p->kv_heads) return -1;
    const size_t smem = (size_t)(p->rot_dims + 8 * p->dim) * sizeof(float);
    if (smem > 48 * 1024) return -1;
    const dim3 grid(T, (p->heads + p->kv_heads + 7) / 8);
    if (out_f32) sl_launch(grouped_pre_kernel<float, float>, grid, 256, smem, s, *p);
    else if (in_f32) sl_launch(grouped_pre_kernel<float, bf16>, grid, 256, smem, s, *p);
    else sl_launch(grouped_pre_kernel<bf16, bf16>, grid, 256, smem, s, *p);
    return SL_LAUNCH_CHECK();
}

SL_API int sl_grouped_row_pre(const GroupedRowPreParams* p, int T, int in_f32, int out_f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->rot_dims > p->dim || p->rot_dims % 2 != 0 || (out_f32 && !in_f32) || (p->v_turn != nullptr && p->vdim % 2 != 0)) return -1;
    const size_t smem = (size_t)(p->heads + p->kv_heads) * p->dim * sizeof(float);
    if (smem > 200 * 1024) return -1;
    const uintptr_t at = (uintptr_t)p->q | (uintptr_t)p->k | (uintptr_t)p->v;
    auto pieces = [&](int vw) { return p->dim % vw == 0 && p->vdim % vw == 0 && p->ld % vw == 0 && at % (vw == 8 ? 16 : vw * (in_f32 ? 4 : 2)) == 0; };
    const int vw = pieces(8) ? 8 : pieces(2) ? 2 : 1;
    // few rows: a thread takes one piece of the row where it can
    const int threads = T > 148 ? (vw == 8 ? 128 : 256) : max(128, min(1024, (p->heads * p->dim / vw + 31) / 32 * 32));
#define SL_RP(VW, TI, TO)                                                                                              \
    {                                                                                                                  \
        auto kern = grouped_row_pre_kernel<VW, TI, TO>;                                                                \
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);      \
        sl_launch(kern, T, threads, smem, s, *p);                                                                      \
    }
    if (out_f32) {
        if (vw == 8) SL_RP(8, float, float) else if (vw == 2) SL_RP(2, float, float) else SL_RP(1, float, float)
    } else if (in_f32) {
        if (vw == 8) SL_RP(8, float, bf16) else if (vw == 2) SL_RP(2, float, bf16) else SL_RP(1, float, bf16)
    } else {
        if (vw == 8) SL_RP(8, bf16, bf16) else if (vw == 2) SL_RP(2, bf16, bf16) else SL_RP(1, bf16, bf16)
    }
#undef SL_RP
    return SL_LAUNCH_CHECK();
}

// out [T, 2]: see row_sums_kernel (the norms, angles, caches and q_out of `p` are not read)
SL_API int sl_grouped_row_sums(const GroupedRowPreParams* p, float* out, int T, int in_f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (in_f32) sl_launch(row_sums_kernel<float>, T, 256, 0, s, out, *p);
    else sl_launch(row_sums_kernel<bf16>, T, 256, 0, s, out, *p);
    return SL_LAUNCH_CHECK();
}

SL_API int sl_grouped_rows(const GroupedAttnParams* p, int T, int f32, cudaStream_t s) {
    if (T == 0) return 0;
    if (p->vdim > 128 * ROWS_MAXV || (p->turn != nullptr && p->vdim % 2 != 0) || T > 65535 || p->heads % p->kv_heads != 0) return -1;
    const size_t smem = (size_t)p->dim * sizeof(float);
    if (smem > 40 * 1024) return -1;
    if (f32) sl_launch(grouped_rows_kernel<float>, dim3(p->heads, T), 128, smem, s, *p);
    else sl_launch(grouped_rows_kernel<bf16>, dim3(p->heads, T), 128, smem, s, *p);
    return SL_LAUNCH_CHECK();
}

// 1 when the tensor-core decode kernel takes these sizes.
SL_API int sl_grouped_decode_ok(int dim, int vdim) {
    return dim >= 8 && vdim >= 8 && dim % 8 == 0 && vdim % 8 == 0 && dim <= 256 && vdim <= 256 && decode_smem(dim, vdim) <= 200 * 1024;
}

SL_API int sl_grouped_decode(const GroupedAttnParams* p, int T, cudaStream_t s) {
    if (T == 0) return 0;
    if (!sl_grouped_decode_ok(p->dim, p->vdim) || p->splits < 1 || p->splits > 64 || T > 65535 || p->heads % p->kv_heads != 0) return -1;
    if (p->ldo % 2 != 0 || (p->splits > 1 && (p->o_part == nullptr || p->lse_part == nullptr))) return -1;
    const size_t smem = decode_smem(p->dim, p->vdim);
    const dim3 grid(p->splits, p->kv_heads * ((p->heads / p->kv_heads + 15) / 16), T);
#define SL_GD(NTW)                                                                                                      \
    {                                                                                                                   \
        auto kern = grouped_decode_kernel<NTW>;                                                                         \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                             \
        sl_launch(kern, grid, DT, smem, s, *p);                                                                         \
    }
    if (p->vdim <= 64) SL_GD(2) else if (p->vdim <= 128) SL_GD(4) else SL_GD(8)
#undef SL_GD
    if (p->splits > 1) sl_launch(grouped_merge_kernel, dim3(p->heads, T), 64, 0, s, *p);
    return SL_LAUNCH_CHECK();
}
