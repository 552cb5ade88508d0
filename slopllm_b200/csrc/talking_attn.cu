// Talking heads over a paged cache: grouped-query attention whose query heads' scores are mixed before the softmax,
//
//   s_h[j] = sum_g talk[h, g] * scale * q_g . k_j[key head of g],      o_h = softmax_j(s_h[j]) . v_j[value head of h],
//
// with positions that see their own chunk of the sequence only.
//
//  * talking_rows_kernel: independent token rows on the CUDA cores, any sizes, bf16 or fp32.
//  * talking_mma_kernel: portions of prompts (up to 16 queries per CTA) and decoding (one), all heads in one CTA, on the tensor cores.
//    Per tile of keys:  (1) every key head's scores, a 16-row block of (head of the group, query) rows per warp, left in shared memory as
//    two bf16 terms, hi + lo;  (2) the mixture as a second product, talk x scores, one query and 16 output heads per warp, whose result
//    holds all keys of the tile for a row: mask and online softmax in registers, weights back to shared memory as hi + lo;  (3) the
//    weighted values, accumulated in registers by the warps of (1).  Key rows and value rows (all heads of a token are neighbours in the
//    cache) come by one bulk copy each, the next tile's keys during (2) and (3), its values during (1) and (2).
//  * talking_merge_kernel: joins the key splits of few queries.
//
// Scores and weights lie in blocks of eight keys: [head][key block][query][8 keys], so that a block is one 16-byte row of every matrix
// that is loaded from there, by query rows (3) as well as by head rows (2).
#include "common.cuh"
#include "mma_sync.cuh"
#include "tcgen05.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

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
    const int4* tiles;                   // portions: first token, tokens, position of the first, page-table row (null: one token each)
    int splits;
    float *o_part, *lse_part;            // [T, out_heads, splits, vdim], [T, out_heads, splits] (more than one split)
    int* err;
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

// ---- tensor-core form ----------------------------------------------------------------------------------------------------

constexpr int WARPS = 16, MAX_SMEM = 232448;

struct MmaPlan {
    int bq, kt;                          // queries per CTA, keys per tile (0: the sizes do not fit)
    int mt;                              // 16-row blocks of a key head's (head, query) rows
    int ldq, q_swz;                      // bytes of a query row; its 16-byte pieces are permuted by the row's low bits
    int ldk, ldv;                        // bytes of a key / value row
    int wpv, per_v;                      // warps of a value unit, its 8-wide value tiles per warp
    int smem, k_at, v_at, s_at, f_at;
};

// Bytes of a head's scores (one plane).  Their 16-byte pieces are permuted by the head's low bits where that stays inside.
__host__ __device__ constexpr int score_swizzle(int kt, int bq) { return kt / 8 * bq % 8 == 0 ? 7 : 0; }
__host__ __device__ constexpr int score_bytes(int kt, int bq) { return kt / 8 * bq * 16 + (score_swizzle(kt, bq) ? 0 : 16); }

MmaPlan make_plan(int heads, int kv_heads, int out_heads, int v_heads, int dim, int vdim, bool decode) {
    MmaPlan best = {};
    const int r = heads / kv_heads;
    if (dim % 8 != 0 || vdim % 8 != 0 || heads > 64 || heads % kv_heads != 0 || out_heads != v_heads * r || out_heads > heads) return best;
    const int dqp = (dim + 15) / 16 * 16, krow = kv_heads * dim * 2, vrow = v_heads * vdim * 2, mto = (out_heads + 15) / 16;
    const int hp = heads <= 16 ? 16 : heads <= 32 ? 32 : 64;      // (of the kernel's instances)
    for (int bq = decode ? 1 : 16; bq >= 1; bq = bq > 4 ? bq / 2 : bq - 3)      // 16, 8, 4, 1
        for (int kt = 64; kt >= 16; kt /= 2) {
            MmaPlan m = {};
            m.bq = bq; m.kt = kt;
            m.mt = (r * bq + 15) / 16;
            const int units = v_heads * m.mt;
            if (units > WARPS || bq * mto > WARPS || bq * hp > 256) continue;
            m.wpv = WARPS / units;
            m.per_v = ((vdim / 8 + m.wpv - 1) / m.wpv + 1) / 2 * 2;
            if (m.per_v > 16 || (kt == 64 && m.per_v > 8)) continue;
            m.q_swz = dqp % 64 == 0 ? 7 : 0;
            m.ldq = dqp * 2 + (m.q_swz ? 0 : 16);
            m.ldk = krow + (krow / 16 % 2 == 0 ? 16 : dim % 16 != 0 ? 32 : 0);
            m.ldv = vrow + (vrow / 16 % 2 == 0 ? 16 : 0);
            m.k_at = kv_heads * m.mt * 16 * m.ldq;
            m.v_at = m.k_at + kt * m.ldk;
            m.s_at = m.v_at + kt * m.ldv;
            m.f_at = m.s_at + 2 * hp * score_bytes(kt, bq);
            m.smem = m.f_at + out_heads * bq * 4;
            if (m.smem + 64 > MAX_SMEM) continue;
            return m;
        }
    return best;
}

__device__ __forceinline__ float exp2_hw(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void bar_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

constexpr float RAISE = 8.f;             // a row's reference is raised when its maximum has grown by more than 2^8

// grid (splits, tiles), block 512.  KT keys per tile, up to NVT 8-wide value tiles per warp, up to 16 * HT heads, BQ queries.
template <int KT, int NVT, int HT, int BQ>
__global__ void __launch_bounds__(WARPS * 32, 1) talking_mma_kernel(TalkingParams p, MmaPlan m) {
    pdl_grid_sync();
    extern __shared__ __align__(128) unsigned char smraw[];
    __shared__ __align__(8) uint64_t bars[2];                       // keys, values have arrived
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, c4 = lane & 3;
    constexpr int LDS = score_bytes(KT, BQ), SWZ = score_swizzle(KT, BQ), HP = HT * 16, PLANE = HP * LDS;
    const int r = p.heads / p.kv_heads, rows = r * BQ, unit_rows = m.mt * 16;
    unsigned char *qs = smraw, *ks = smraw + m.k_at, *vs = smraw + m.v_at, *sh = smraw + m.s_at;
    float* fac = reinterpret_cast<float*>(smraw + m.f_at);          // [out_heads][BQ]
    int4 tile;
    if (p.tiles != nullptr) {
        tile = p.tiles[blockIdx.y];
    } else {
        tile = make_int4(blockIdx.y, 1, p.positions[blockIdx.y], p.batch_idx[blockIdx.y]);
    }
    const int tok = tile.x, count = tile.y, pos0 = tile.z, split = blockIdx.x;
    const int lo = p.chunk > 0 ? pos0 / p.chunk * p.chunk : 0, end = pos0 + count;
    const int tiles = (end - lo + KT - 1) / KT, per = (tiles + p.splits - 1) / p.splits;
    const int tb = min(tiles, split * per), te = min(tiles, tb + per);
    const int* pt = p.page_table + (size_t)tile.w * p.pt_stride;
    const uint32_t krow = p.kv_heads * p.dim * 2, vrow = p.v_heads * p.vdim * 2;

    // warp 0: pages of this lane's keys of tile j, and the keys' cache slots (behind the last key: the last once more, never visible)
    constexpr int KPL = (KT + 31) / 32;                              // keys per lane
    auto key_of = [&](int j, int i) { return min(lo + j * KT + i * 32 + lane, end - 1); };
    auto pages_of = [&](int j, int (&page)[KPL]) {
#pragma unroll
        for (int i = 0; i < KPL; ++i) page[i] = pt[key_of(j, i) / p.page_size];
    };
    auto slots_of = [&](int j, const int (&page)[KPL], long long (&slot)[KPL]) {
#pragma unroll
        for (int i = 0; i < KPL; ++i) {
            const long long s = (long long)page[i] * p.page_size + key_of(j, i) % p.page_size;
            slot[i] = guard_ok(p.guard, 32, s, p.num_slots) ? s : 0;
        }
    };
    auto fetch = [&](unsigned char* dst, int ld, const void* cache, uint32_t row, uint64_t* bar, const long long (&slot)[KPL]) {
        if (lane == 0) tc::mbar_expect_tx(bar, KT * row);
        __syncwarp();
#pragma unroll
        for (int i = 0; i < KPL; ++i)
            if (lane < KT) tc::bulk_load_1d(dst + (i * 32 + lane) * ld, (const unsigned char*)cache + (size_t)slot[i] * row, row, bar);
    };
    if (tid == 0) {
        tc::mbar_init(&bars[0], 1);
        tc::mbar_init(&bars[1], 1);
        tc::mbar_fence_init();
        tc::fence_proxy_async_smem();
    }
    long long slot[KPL] = {};
    int page_next[KPL] = {};
    if (warp == 0) {
        __syncwarp();
        if (tb < te) {
            pages_of(tb, page_next);
            slots_of(tb, page_next, slot);
            fetch(ks, m.ldk, p.k_cache, krow, &bars[0], slot);
        }
    }
    // queries, zeros behind the last row and the last value; zeros in the scores of heads that are not there
    const int dp = (p.dim + 15) / 16 * 2;
    for (int i = tid; i < p.kv_heads * unit_rows * dp; i += WARPS * 32) {
        const int row = i / dp, c = i - row * dp, unit = row / unit_rows, rho = row - unit * unit_rows, g = rho / BQ, qi = rho % BQ;
        uint4 x = make_uint4(0, 0, 0, 0);
        if (rho < rows && qi < count && c * 8 < p.dim)
            x = *reinterpret_cast<const uint4*>((const bf16*)p.q + ((size_t)(tok + qi) * p.heads + unit * r + g) * p.dim + c * 8);
        *reinterpret_cast<uint4*>(qs + row * m.ldq + ((c ^ (row & m.q_swz)) << 4)) = x;
    }
    for (int i = tid; i < 2 * PLANE / 16; i += WARPS * 32) *reinterpret_cast<uint4*>(sh + i * 16) = make_uint4(0, 0, 0, 0);
    if (p.dim % 16 != 0)                                            // (the last head's 16-value steps reach into the padding)
        for (int i = tid; i < KT; i += WARPS * 32) *reinterpret_cast<uint4*>(ks + i * m.ldk + krow) = make_uint4(0, 0, 0, 0);
    // the mixture: this warp's query and 16 output heads
    const int mto = (p.out_heads + 15) / 16, qi_mix = warp / mto, h_mix = (warp - qi_mix * mto) * 16;
    const bool mixes = qi_mix < count;                              // (qi_mix < BQ follows)
    uint32_t tf[HT][4];
#pragma unroll
    for (int k = 0; k < HT; ++k)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int h = h_mix + g8 + (i & 1) * 8, g = k * 16 + (i >> 1) * 8 + c4 * 2;
            float a = 0.f, b = 0.f;
            if (mixes && h < p.out_heads) {
                a = g < p.heads ? p.talk[h * p.heads + g] : 0.f;
                b = g + 1 < p.heads ? p.talk[h * p.heads + g + 1] : 0.f;
            }
            tf[k][i] = f2_to_bf162(a, b);
        }
    const int q_pos = pos0 + qi_mix, q_lo = p.chunk > 0 ? q_pos / p.chunk * p.chunk : 0;
    const float scale_log2 = p.scale * LOG2E;
    float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
    // the values: this warp's unit and value tiles
    const int uv = warp / m.wpv, n0 = (warp - uv * m.wpv) * m.per_v, nn = uv < p.v_heads * m.mt ? min(m.per_v, p.vdim / 8 - n0) : 0;
    const int hv = uv / m.mt, rv = (uv - hv * m.mt) * 16;           // value head, first of the unit's rows
    float acc[NVT][4];
#pragma unroll
    for (int i = 0; i < NVT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    // the row of weights that this lane addresses
    const int a_rho = min(rv + (lane & 15), rows - 1), a_head = min(hv * r + a_rho / BQ, p.out_heads - 1), a_qi = a_rho % BQ;
    const int units_k = p.kv_heads * m.mt;
    const int wpq = KT >= 64 && units_k * 4 <= WARPS ? 4 : KT >= 32 && units_k * 2 <= WARPS ? 2 : 1, keys_w = KT / wpq;      // warps of a unit, keys of each
    auto s_off = [&](int h, int kb, int qi) { return h * LDS + (((kb * BQ + qi) ^ (h & SWZ)) << 4); };
    const int u_first = warp / wpq, kh_first = u_first / m.mt;
    bool v_row[2];                                                  // this thread's rows of the unit are those of a query
#pragma unroll
    for (int e = 0; e < 2; ++e) v_row[e] = rv + g8 + e * 8 < rows && (rv + g8 + e * 8) % BQ < count;

    __syncthreads();
    bool bad = false;
    for (int j = tb; j < te; ++j) {
        const uint32_t parity = (j - tb) & 1;
        if (__syncthreads_or(!tc::mbar_wait(&bars[0], parity))) { bad = true; break; }
        if (warp == 0) fetch(vs, m.ldv, p.v_cache, vrow, &bars[1], slot);
        if (warp == 0 && j + 1 < te) pages_of(j + 1, page_next);
        // (1) scores
        for (int i = warp; i < units_k * wpq; i += WARPS) {
            const int u = i == warp ? u_first : i / wpq, kh = i == warp ? kh_first : u / m.mt, r0 = (u - kh * m.mt) * 16;
            const int qr = kh * unit_rows + r0 + (lane & 15);
            const unsigned char* qrow = qs + qr * m.ldq;
#pragma unroll
            for (int x = 0; x < KT; x += 32) {                      // 32 keys (16 if the warp has no more)
                if (x > 0 && x >= keys_w) break;
                const int kb0 = (i - u * wpq) * keys_w + x;         // first key
                const bool both = KT > 16 && x + 16 < keys_w;
                float s[4][4] = {};
                const unsigned char* krow_s = ks + (kb0 + (lane & 7) + (lane >> 4) * 8) * m.ldk + kh * p.dim * 2 + ((lane >> 3) & 1) * 16;
#pragma unroll 4
                for (int c = 0; c < dp; c += 2) {
                    uint32_t a[4], b[4];
                    ldsm_x4(a, qrow + (((c + (lane >> 4)) ^ (qr & m.q_swz)) << 4));
                    ldsm_x4(b, krow_s + c * 16);
                    mma_bf16_16816(s[0], a, b[0], b[1]);
                    mma_bf16_16816(s[1], a, b[2], b[3]);
                    if (both) {
                        ldsm_x4(b, krow_s + 16 * m.ldk + c * 16);
                        mma_bf16_16816(s[2], a, b[0], b[1]);
                        mma_bf16_16816(s[3], a, b[2], b[3]);
                    }
                }
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int rho = r0 + g8 + e * 8;
                    if (rho >= rows) continue;
                    const int qi = rho % BQ, h = kh * r + rho / BQ;
#pragma unroll
                    for (int n = 0; n < 4; ++n) {
                        if (n >= 2 && !both) break;
                        uint32_t hi, low;
                        split_bf162(s[n][e * 2], s[n][e * 2 + 1], hi, low);
                        unsigned char* at = sh + s_off(h, kb0 / 8 + n, qi) + c4 * 4;
                        *reinterpret_cast<uint32_t*>(at) = hi;
                        *reinterpret_cast<uint32_t*>(at + PLANE) = low;
                    }
                }
            }
        }
        __syncthreads();
        if (warp == 0 && j + 1 < te) {
            slots_of(j + 1, page_next, slot);
            fetch(ks, m.ldk, p.k_cache, krow, &bars[0], slot);
        }
        // (2) mixture, mask, softmax
        if (mixes) {
            float c[KT / 8][4] = {};
            const int hr = (lane & 7) + ((lane >> 3) & 1) * 8;
#pragma unroll
            for (int k = 0; k < HT; ++k)
#pragma unroll
                for (int n = 0; n < KT / 8; n += 2) {
                    uint32_t b[4];
                    const unsigned char* at = sh + s_off(k * 16 + hr, n + (lane >> 4), qi_mix);
                    ldsm_x4_trans(b, at);
                    mma_bf16_16816(c[n], tf[k], b[0], b[1]);
                    mma_bf16_16816(c[n + 1], tf[k], b[2], b[3]);
                    ldsm_x4_trans(b, at + PLANE);
                    mma_bf16_16816(c[n], tf[k], b[0], b[1]);
                    mma_bf16_16816(c[n + 1], tf[k], b[2], b[3]);
                }
            if (mto > 1) bar_sync(1 + qi_mix, mto * 32);            // (the weights take the scores' place)
            else __syncwarp();
            const int k_first = lo + j * KT, key0 = k_first + c4 * 2;
#pragma unroll
            for (int n = 0; n < KT / 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) c[n][e] *= scale_log2;
            if (k_first < q_lo || k_first + KT - 1 > q_pos) {       // (a tile inside the query's chunk is seen whole)
#pragma unroll
                for (int n = 0; n < KT / 8; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int key = key0 + n * 8 + (e & 1);
                        if (key < q_lo || key > q_pos) c[n][e] = -INFINITY;
                    }
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float top = mx[e];
#pragma unroll
                for (int n = 0; n < KT / 8; ++n) top = fmaxf(top, fmaxf(c[n][e * 2], c[n][e * 2 + 1]));
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 1));
                top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, 2));
                if (top <= mx[e] + RAISE) top = mx[e];
                const float base = top == -INFINITY ? 0.f : top, f = exp2_hw(mx[e] - base);
                const int h = h_mix + g8 + e * 8;
                float l = 0.f;
#pragma unroll
                for (int n = 0; n < KT / 8; ++n) {
                    const float x = exp2_hw(c[n][e * 2] - base), y = exp2_hw(c[n][e * 2 + 1] - base);
                    l += x + y;
                    if (h < p.out_heads) {
                        uint32_t hi, low;
                        split_bf162(x, y, hi, low);
                        unsigned char* at = sh + s_off(h, n, qi_mix) + c4 * 4;
                        *reinterpret_cast<uint32_t*>(at) = hi;
                        *reinterpret_cast<uint32_t*>(at + PLANE) = low;
                    }
                }
                sum[e] = sum[e] * f + l;
                mx[e] = top;
                if (c4 == 0 && h < p.out_heads) fac[h * BQ + qi_mix] = f;
            }
        }
        if (__syncthreads_or(!tc::mbar_wait(&bars[1], parity))) { bad = true; break; }
        // (3) values
        if (nn > 0) {
            float f[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) f[e] = v_row[e] ? fac[hv * rows + rv + g8 + e * 8] : 1.f;
            if (__any_sync(0xffffffffu, f[0] != 1.f || f[1] != 1.f)) {
#pragma unroll
                for (int i = 0; i < NVT; ++i) { acc[i][0] *= f[0]; acc[i][1] *= f[0]; acc[i][2] *= f[1]; acc[i][3] *= f[1]; }
            }
#pragma unroll
            for (int k = 0; k < KT / 16; ++k) {
                uint32_t a[4], al[4];
                const unsigned char* at = sh + s_off(a_head, k * 2 + (lane >> 4), a_qi);
                ldsm_x4(a, at);
                ldsm_x4(al, at + PLANE);
                const unsigned char* v_at = vs + (k * 16 + (lane & 15)) * m.ldv + (hv * p.vdim + n0 * 8) * 2;
                auto pair = [&](int i) {
                    uint32_t b[4];
                    ldsm_x4_trans(b, v_at + (lane >> 4) * 16 + i * 16);
                    mma_bf16_16816(acc[i], a, b[0], b[1]);
                    mma_bf16_16816(acc[i + 1], a, b[2], b[3]);
                    mma_bf16_16816(acc[i], al, b[0], b[1]);
                    mma_bf16_16816(acc[i + 1], al, b[2], b[3]);
                };
                if (nn == NVT) {
#pragma unroll
                    for (int i = 0; i < NVT; i += 2) pair(i);
                } else {
#pragma unroll
                    for (int i = 0; i < NVT; i += 2) {
                        if (i >= nn) break;
                        if (i + 1 < nn) {
                            pair(i);
                        } else {
                            uint32_t b[2];
                            ldsm_x2_trans(b[0], b[1], v_at + i * 16);
                            mma_bf16_16816(acc[i], a, b[0], b[1]);
                            mma_bf16_16816(acc[i], al, b[0], b[1]);
                        }
                    }
                }
            }
        }
    }
    if (bad) {                                                      // an expired wait: nothing more is started, copies in flight are let in
        if (tid == 0) {
            p.err[0] = 33;
            tc::mbar_wait(&bars[0], 0, 100000000ull);
            tc::mbar_wait(&bars[0], 1, 100000000ull);
            tc::mbar_wait(&bars[1], 0, 100000000ull);
            tc::mbar_wait(&bars[1], 1, 100000000ull);
        }
        return;
    }
    __syncthreads();
    if (mixes) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 1);
            sum[e] += __shfl_xor_sync(0xffffffffu, sum[e], 2);
            const int h = h_mix + g8 + e * 8;
            if (c4 == 0 && h < p.out_heads) {
                fac[h * BQ + qi_mix] = sum[e] > 0.f ? 1.f / sum[e] : 0.f;
                if (p.splits > 1)
                    p.lse_part[((size_t)(tok + qi_mix) * p.out_heads + h) * p.splits + split] = sum[e] > 0.f ? (mx[e] + log2f(sum[e])) / LOG2E : -INFINITY;
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int rho = rv + g8 + e * 8, qi = rho % BQ, h = hv * r + rho / BQ;
        if (nn <= 0 || !v_row[e]) continue;
        const float inv = fac[h * BQ + qi];
#pragma unroll
        for (int i = 0; i < NVT; ++i) {
            if (i >= nn) break;
            const int d = (n0 + i) * 8 + c4 * 2;
            const float x = acc[i][e * 2] * inv, y = acc[i][e * 2 + 1] * inv;
            if (p.splits == 1) *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)(tok + qi) * p.ldo + (size_t)h * p.vdim + d) = f2_to_bf162(x, y);
            else *reinterpret_cast<float2*>(p.o_part + (((size_t)(tok + qi) * p.out_heads + h) * p.splits + split) * p.vdim + d) = make_float2(x, y);
        }
    }
}

// grid (out_heads, T), block 64: two values per thread and pass
__global__ void __launch_bounds__(64) talking_merge_kernel(TalkingParams p) {
    pdl_grid_sync();
    __shared__ float w[64];
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
    const size_t row = (size_t)t * p.out_heads + h;
    const float a = lane < p.splits ? p.lse_part[row * p.splits + lane] : -INFINITY;
    const float b = lane + 32 < p.splits ? p.lse_part[row * p.splits + lane + 32] : -INFINITY;
    const float top = warp_max(fmaxf(a, b));
    const float ea = a == -INFINITY ? 0.f : expf(a - top), eb = b == -INFINITY ? 0.f : expf(b - top);
    const float inv = 1.f / warp_sum(ea + eb);
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
        *reinterpret_cast<uint32_t*>((bf16*)p.out + (size_t)t * p.ldo + (size_t)h * p.vdim + d) = f2_to_bf162(x, y);
    }
}

template <int KT, int NVT>
int launch_mma(const TalkingParams* p, const MmaPlan& m, int tiles, cudaStream_t s) {
    auto go = [&](auto kern) {
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, m.smem);
        sl_launch(kern, dim3(p->splits, tiles), WARPS * 32, m.smem, s, *p, m);
        return SL_LAUNCH_CHECK();
    };
    const int ht = (p->heads + 15) / 16;
    if (ht == 1) {
        if (m.bq == 16) return go(talking_mma_kernel<KT, NVT, 1, 16>);
        if (m.bq == 8) return go(talking_mma_kernel<KT, NVT, 1, 8>);
        return m.bq == 4 ? go(talking_mma_kernel<KT, NVT, 1, 4>) : go(talking_mma_kernel<KT, NVT, 1, 1>);
    }
    if (ht == 2) {
        if (m.bq == 8) return go(talking_mma_kernel<KT, NVT, 2, 8>);
        return m.bq == 4 ? go(talking_mma_kernel<KT, NVT, 2, 4>) : go(talking_mma_kernel<KT, NVT, 2, 1>);
    }
    return m.bq == 4 ? go(talking_mma_kernel<KT, NVT, 4, 4>) : go(talking_mma_kernel<KT, NVT, 4, 1>);
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

// Queries per CTA of the tensor-core kernel (decode: 1), 0 when it does not take these sizes.
SL_API int sl_talking_queries(int heads, int kv_heads, int out_heads, int v_heads, int dim, int vdim, int decode) {
    if (heads < 1 || kv_heads < 1 || v_heads < 1 || dim < 8 || vdim < 8) return 0;
    return make_plan(heads, kv_heads, out_heads, v_heads, dim, vdim, decode != 0).bq;
}

// Keys per tile, as above.
SL_API int sl_talking_keys(int heads, int kv_heads, int out_heads, int v_heads, int dim, int vdim, int decode) {
    if (heads < 1 || kv_heads < 1 || v_heads < 1 || dim < 8 || vdim < 8) return 0;
    return make_plan(heads, kv_heads, out_heads, v_heads, dim, vdim, decode != 0).kt;
}

// `tiles` query tiles (without p->tiles: tokens) of T tokens.
SL_API int sl_talking_mma(const TalkingParams* p, int tiles, int T, cudaStream_t s) {
    if (T == 0 || tiles == 0) return 0;
    if (!shape_ok(p) || p->dim < 8 || p->vdim < 8 || p->splits < 1 || p->splits > 64 || tiles > 65535 || T > 65535 || p->ldo % 2 != 0 || p->err == nullptr) return -1;
    if (p->splits > 1 && (p->o_part == nullptr || p->lse_part == nullptr)) return -1;
    if (((uintptr_t)p->q | (uintptr_t)p->k_cache | (uintptr_t)p->v_cache) % 16 != 0) return -1;
    const MmaPlan m = make_plan(p->heads, p->kv_heads, p->out_heads, p->v_heads, p->dim, p->vdim, p->tiles == nullptr);
    if (m.bq == 0) return -1;
    int rc;
#define SL_TM(KT) (m.per_v <= 8 ? launch_mma<KT, 8>(p, m, tiles, s) : launch_mma<KT, 16>(p, m, tiles, s))
    rc = m.kt == 64 ? launch_mma<64, 8>(p, m, tiles, s) : m.kt == 32 ? SL_TM(32) : SL_TM(16);
#undef SL_TM
    if (rc == 0 && p->splits > 1) {
        sl_launch(talking_merge_kernel, dim3(p->out_heads, T), 64, 0, s, *p);
        rc = SL_LAUNCH_CHECK();
    }
    return rc;
}
