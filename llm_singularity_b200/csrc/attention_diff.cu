// Differential attention over the paged cache: every head attends twice to the same values, each time
// with a query and a key of its own ("map" 0 and 1), and what leaves is the difference:
//
//   o   = a_0 - lambda a_1          a_m = softmax(scale q_m . k_m) v, over the keys the row sees
//   out = o / sqrt(mean(o^2) + eps) * post          over the head's dv values
//
// lambda is one 32-bit number on the device (a layer's own), post a constant.  A query row's queries
// are [map 0 | map 1] of dk each, a cached key [map 0 | map 1] likewise, [page][kv head][offset][2 dk];
// values are [page][kv head][offset][dv].  Which keys a row sees (causal, window, chunk), how query
// heads share kv heads and how rows are numbered is as in attention_dv.cu.  Scores, weights, sums, the
// difference and the norm are 32-bit; a_0 and a_1 are never rounded.
//
// Generic form (any sizes, 32-bit or bfloat16 storage): one warp owns a (row, head) and walks the keys
// once for both maps.
//
// Tensor-core form (bfloat16, dk and dv multiples of 8, dk up to 128 and dv up to 256): a block owns a
// request, a kv head and 64 rows; four warps work on map 0 and four on map 1 of the same rows, on the
// same tiles of keys and values in shared memory (mma.sync m16n8k16, cp.async ring).  Map 1's warps
// leave their normalized rows in shared memory, map 0's take the difference and the norm.  Steps whose
// requests bring at most 16 rows each get blocks of 16 rows, the four warps of a map dealing the keys of
// a tile among themselves; where such blocks are few, a row tile's keys are shared among up to eight
// blocks whose partial sums a second kernel brings together.
#define LSB_CLUSTER_ALONG_X
#include "attention_dv.cuh"

LSB_DEFINE_STATUS()

constexpr int kDiffWarps = 4;              // of the generic form
constexpr int kDiffMaxDim = 512;           // 2 dk and dv of the generic form
constexpr int kDiffThreads = 256;          // of the tensor-core form: four warps a map

struct DiffArgs {
    const void *q, *k_pages, *v_pages;
    const int *q_start, *kv_len, *table_rows, *block_table;
    int table_stride;
    void* out;
    int nh, nkv, dk, dv, page_size, num_pages;
    float scale;
    int window, chunk;
    const float* lambda;
    float eps, post;
};

__device__ __forceinline__ int diff_lowest(int p, int window, int chunk) {
    int lo = (window > 0 && p - window + 1 > 0) ? p - window + 1 : 0;
    if (chunk > 0) lo = max(lo, (p / chunk) * chunk);
    return lo;
}

// ------------------------------------------------------------------ generic form
template <typename T>
__global__ void __launch_bounds__(kDiffWarps * 32) attention_diff_generic_kernel(const DiffArgs a, int vec) {
    __shared__ float q_sh[kDiffWarps][kDiffMaxDim];
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.z, h = blockIdx.y;
    const int qs = a.q_start[r];
    const int q_len = a.q_start[r + 1] - qs;
    const int i = blockIdx.x * kDiffWarps + warp;           // row within the request
    if (i >= q_len) return;                                  // whole warp leaves together
    const int p = a.kv_len[r] - q_len + i;
    const int lo = diff_lowest(p, a.window, a.chunk);
    const int g = h / (a.nh / a.nkv), dk = a.dk, dv = a.dv;
    const size_t t = (size_t)qs + i;
    const int* bt = a.block_table + (size_t)a.table_rows[r] * a.table_stride;
    const T* k_pages = (const T*)a.k_pages;
    const T* v_pages = (const T*)a.v_pages;
    const T* qr = (const T*)a.q + (t * a.nh + h) * (2 * dk);
    for (int d = lane; d < 2 * dk; d += 32) q_sh[warp][d] = lsb_to_float(qr[d]) * a.scale;
    __syncwarp();

    constexpr int kAccs = kDiffMaxDim / 32;
    float acc0[kAccs], acc1[kAccs];
#pragma unroll
    for (int c = 0; c < kAccs; ++c) acc0[c] = acc1[c] = 0.f;
    float m0 = -FLT_MAX, m1 = -FLT_MAX, l0 = 0.f, l1 = 0.f;
    for (int base = lo; base <= p; base += 32) {
        const int kj = base + lane;
        float s0 = -FLT_MAX, s1 = -FLT_MAX;
        long long at = -1;                                   // (page, kv head, offset) as a row number
        if (kj <= p) {
            const int page = bt[kj / a.page_size];
            if (page < 0 || page >= a.num_pages) {
                lsb_set_status(LSB_BAD_PAGE);
            } else {
                at = ((long long)page * a.nkv + g) * a.page_size + (kj % a.page_size);
                const T* kr = k_pages + at * (2 * dk);
                s0 = dv_dot<T>(q_sh[warp], kr, dk, vec != 0);
                s1 = dv_dot<T>(q_sh[warp] + dk, kr + dk, dk, vec != 0);
            }
        }
        const float n0 = fmaxf(m0, lsb_warp_max(s0)), n1 = fmaxf(m1, lsb_warp_max(s1));
        const float c0 = expf(m0 - n0), c1 = expf(m1 - n1);  // (-FLT_MAX first: exp(-huge) = 0)
        const float p0 = at >= 0 ? expf(s0 - n0) : 0.f, p1 = at >= 0 ? expf(s1 - n1) : 0.f;
        l0 = l0 * c0 + lsb_warp_sum(p0);
        l1 = l1 * c1 + lsb_warp_sum(p1);
        m0 = n0;
        m1 = n1;
#pragma unroll
        for (int c = 0; c < kAccs; ++c) {
            acc0[c] *= c0;
            acc1[c] *= c1;
        }
        const int n_valid = min(32, p - base + 1);
        for (int j = 0; j < n_valid; ++j) {
            const float w0 = __shfl_sync(0xffffffffu, p0, j), w1 = __shfl_sync(0xffffffffu, p1, j);
            const long long vat = __shfl_sync(0xffffffffu, at, j);
            if (vat < 0) continue;
            const T* v = v_pages + vat * dv;
#pragma unroll
            for (int c = 0; c < kAccs; ++c) {
                const int d = lane + 32 * c;
                if (d < dv) {
                    const float x = lsb_to_float(v[d]);
                    acc0[c] += w0 * x;
                    acc1[c] += w1 * x;
                }
            }
        }
    }
    const float i0 = l0 > 0.f ? 1.f / l0 : 0.f, i1 = (l1 > 0.f ? 1.f / l1 : 0.f) * a.lambda[0];
    float ss = 0.f;
#pragma unroll
    for (int c = 0; c < kAccs; ++c) {
        acc0[c] = acc0[c] * i0 - acc1[c] * i1;
        if (lane + 32 * c < dv) ss += acc0[c] * acc0[c];
    }
    const float mul = a.post / sqrtf(lsb_warp_sum(ss) / (float)dv + a.eps);
    T* o = (T*)a.out + (t * a.nh + h) * dv;
#pragma unroll
    for (int c = 0; c < kAccs; ++c)
        if (lane + 32 * c < dv) o[lane + 32 * c] = lsb_from_float<T>(acc0[c] * mul);
}

// ------------------------------------------------------------------ tensor-core form
template <int DKP, int DVP, int STAGES, bool NARROW>
struct DiffTile {
    static constexpr int KS = 2 * DKP + 8, VS = DVP + 8;    // row strides in elements: 4 words past a multiple of 32
    static constexpr int PS = DVP + 2;                      // a row of partial sums: O, then m and l
    static constexpr int YS = DVP + 4;                      // a row of map 1 on its way to map 0's warps
    static constexpr size_t kRing = (size_t)STAGES * kMmaKeys * (KS + VS) * 2;
    static constexpr size_t kMeet = NARROW ? (size_t)8 * 16 * PS * 4 : (size_t)kMmaRows * YS * 4;
    static constexpr size_t kTotal = kRing > kMeet ? kRing : kMeet;
};

template <int DKP, int DVP, int STAGES, bool NARROW>
__global__ void __launch_bounds__(kDiffThreads)
attention_diff_mma_kernel(const DiffArgs a, float scale_log2, int ksplit, float* __restrict__ scratch) {
    using L = DiffTile<DKP, DVP, STAGES, NARROW>;
    constexpr int KS = L::KS, VS = L::VS;
    typedef __nv_bfloat16 bf16;
    extern __shared__ __align__(16) unsigned char diff_smem[];
    bf16* Ks = reinterpret_cast<bf16*>(diff_smem);          // [STAGES][64][map 0 (DKP) | map 1 (DKP) | 8]
    bf16* Vs = Ks + STAGES * kMmaKeys * KS;                 // [STAGES][64][VS]
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int nh = a.nh, nkv = a.nkv, dk = a.dk, dv = a.dv, page_size = a.page_size;
    const int r = blockIdx.z, g = blockIdx.y, group = nh / nkv;
    const int qs = a.q_start[r];
    const int q_len = a.q_start[r + 1] - qs;
    const int rows_total = q_len * group;
    constexpr int NJ = NARROW ? 2 : 8;                 // blocks of 8 keys a warp takes of a tile
    constexpr int NKK = NARROW ? 1 : 4;                // and the same keys as k-steps of 16
    constexpr int block_rows = NARROW ? 16 : kMmaRows;
    const int row_tile = NARROW ? blockIdx.x / ksplit : blockIdx.x, key_part = NARROW ? blockIdx.x % ksplit : 0;
    const int tile_row0 = row_tile * block_rows;
    if (tile_row0 >= rows_total) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tid4 = lane & 3;
    const int map = warp >> 2, sub = warp & 3;         // which softmax, and which rows (or keys) of it
    const int kv_len = a.kv_len[r];
    const int p_base = kv_len - q_len;
    const int last_row = min(tile_row0 + block_rows, rows_total) - 1;
    const int last_pos = p_base + last_row / group;
    const int key_lo = diff_lowest(p_base + tile_row0 / group, a.window, a.chunk);   // the first key any row of the block sees
    int kt0 = key_lo / kMmaKeys, kt1 = last_pos / kMmaKeys;
    if (NARROW && ksplit > 1) {                        // this block's share of the key tiles (it may be empty)
        const int per = (kt1 - kt0 + ksplit) / ksplit;
        kt0 += key_part * per;
        kt1 = min(kt1, kt0 + per - 1);
    }
    const int* bt = a.block_table + (size_t)a.table_rows[r] * a.table_stride;

    // this thread's two rows (gid and gid + 8 of the warp's slab)
    const int slab = tile_row0 + (NARROW ? 0 : sub * 16);
    const int row_a = slab + gid, row_b = row_a + 8;
    const bool ok_a = row_a < rows_total, ok_b = row_b < rows_total;
    const int pos_a = p_base + row_a / group, pos_b = p_base + row_b / group;
    const int lo_a = diff_lowest(pos_a, a.window, a.chunk), lo_b = diff_lowest(pos_b, a.window, a.chunk);
    const int h_a = g * group + row_a % group, h_b = g * group + row_b % group;
    const size_t t_a = (size_t)qs + row_a / group, t_b = (size_t)qs + row_b / group;

    uint32_t qa[DKP / 16][4];
    {
        const bf16* qa_row = (const bf16*)a.q + (t_a * nh + h_a) * (2 * dk) + map * dk;
        const bf16* qb_row = (const bf16*)a.q + (t_b * nh + h_b) * (2 * dk) + map * dk;
#pragma unroll
        for (int ks = 0; ks < DKP / 16; ++ks) {
            qa[ks][0] = qa[ks][1] = qa[ks][2] = qa[ks][3] = 0u;
            const int c = ks * 16 + 2 * tid4;
            if (ks * 16 < dk) {
                if (ok_a) qa[ks][0] = *reinterpret_cast<const uint32_t*>(qa_row + c);
                if (ok_b) qa[ks][1] = *reinterpret_cast<const uint32_t*>(qb_row + c);
            }
            if (ks * 16 + 8 < dk) {
                if (ok_a) qa[ks][2] = *reinterpret_cast<const uint32_t*>(qa_row + c + 8);
                if (ok_b) qa[ks][3] = *reinterpret_cast<const uint32_t*>(qb_row + c + 8);
            }
        }
    }
    float o[DVP / 8][4];
#pragma unroll
    for (int nb = 0; nb < DVP / 8; ++nb) o[nb][0] = o[nb][1] = o[nb][2] = o[nb][3] = 0.f;
    float m_a = -FLT_MAX, m_b = -FLT_MAX, l_a = 0.f, l_b = 0.f;

    // Loading: four threads own a key row of a tile (key chunks of both maps, value chunks, 16 bytes each).
    // The row's place in the pages is looked up one tile ahead of the copies that need it.
    const int my_row = threadIdx.x >> 2, my_part = threadIdx.x & 3;
    constexpr int kNoRow = -2, kPastEnd = -1;          // a page id a request never holds / nothing to load
    auto place = [&](int kt) -> int {
        const int kj = kt * kMmaKeys + my_row;
        // (keys behind every row's window are never looked up: their pages may have gone back to the pool)
        if (kt > kt1 || kj > last_pos || kj < key_lo) return kPastEnd;
        const int page = bt[kj / page_size];
        return page < 0 ? kNoRow : page;
    };
    const int kper = dk >> 3, vper = dv >> 3;
    auto load_tile = [&](int page, int kt, int buf) {
        long long at = -1;
        if (page >= a.num_pages || page == kNoRow) lsb_set_status(LSB_BAD_PAGE);
        else if (page >= 0) at = ((long long)page * nkv + g) * page_size + ((kt * kMmaKeys + my_row) % page_size);
        bf16* kd = Ks + (buf * kMmaKeys + my_row) * KS;
        bf16* vd = Vs + (buf * kMmaKeys + my_row) * VS;
        const bool real = at >= 0;
        const bf16* ksrc = (const bf16*)a.k_pages + (real ? at * (2 * dk) : 0);
        const bf16* vsrc = (const bf16*)a.v_pages + (real ? at * dv : 0);
#pragma unroll 4
        for (int c = my_part; c < kper; c += 4) {
            dv_cp_async16(kd + c * 8, ksrc + (real ? c * 8 : 0), real);
            dv_cp_async16(kd + DKP + c * 8, ksrc + (real ? dk + c * 8 : 0), real);
        }
#pragma unroll 4
        for (int c = my_part; c < vper; c += 4) dv_cp_async16(vd + c * 8, vsrc + (real ? c * 8 : 0), real);
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    const bool active = NARROW || slab < rows_total;   // a warp whose slab lies past the rows only helps loading
    // the padding of the key and value rows is zeroed once; copies never touch it
    for (int idx = threadIdx.x; idx < STAGES * kMmaKeys; idx += kDiffThreads) {
        for (int c = dk; c < DKP; ++c) Ks[idx * KS + c] = Ks[idx * KS + DKP + c] = __float2bfloat16_rn(0.f);
        for (int c = dv; c < DVP; ++c) Vs[idx * VS + c] = __float2bfloat16_rn(0.f);
    }
    // a group of copies is committed for every tile slot, real or not, so that the count the wait
    // names is the same in every turn of the loop
#pragma unroll
    for (int st = 0; st < STAGES - 1; ++st) {
        if (kt0 + st <= kt1) load_tile(place(kt0 + st), kt0 + st, st);
        else asm volatile("cp.async.commit_group;" ::: "memory");
    }
    int at_next = place(kt0 + STAGES - 1);
    const int slab_lo = diff_lowest(p_base + min(slab + 15, rows_total - 1) / group, a.window, a.chunk);
    const int slab_hi = p_base + slab / group;
    const bool slab_full = slab + 15 < rows_total;
    for (int kt = kt0; kt <= kt1; ++kt) {
        const int buf = (kt - kt0) % STAGES;
        if (kt + STAGES - 1 <= kt1) load_tile(at_next, kt + STAGES - 1, (kt - kt0 + STAGES - 1) % STAGES);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        at_next = place(kt + STAGES);
        asm volatile("cp.async.wait_group %0;" ::"n"(STAGES - 1) : "memory");
        __syncthreads();
        if (active) {
            const int key0 = NARROW ? sub * 16 : 0;            // this warp's first key of the tile
            const bf16* kb = Ks + (buf * kMmaKeys + key0) * KS + map * DKP;
            const bf16* vb = Vs + (buf * kMmaKeys + key0) * VS;
            float s[NJ][4];
#pragma unroll
            for (int j = 0; j < NJ; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < DKP / 16; ++ks) {
#pragma unroll
                for (int j = 0; j < NJ; ++j) {
                    const bf16* krow = kb + (j * 8 + gid) * KS + 2 * tid4 + ks * 16;
                    dv_mma_16816(s[j], qa[ks], *reinterpret_cast<const uint32_t*>(krow),
                                 *reinterpret_cast<const uint32_t*>(krow + 8));
                }
            }
            const int tile_key0 = kt * kMmaKeys + key0;
            const bool interior = slab_full && tile_key0 >= slab_lo && tile_key0 + NJ * 8 - 1 <= slab_hi;
            float mx_a = -FLT_MAX, mx_b = -FLT_MAX;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = tile_key0 + j * 8 + 2 * tid4 + (e & 1);
                    const bool ok = interior || (e < 2 ? (ok_a && key >= lo_a && key <= pos_a)
                                                       : (ok_b && key >= lo_b && key <= pos_b));
                    s[j][e] = ok ? s[j][e] * scale_log2 : -FLT_MAX;
                }
                mx_a = fmaxf(mx_a, fmaxf(s[j][0], s[j][1]));
                mx_b = fmaxf(mx_b, fmaxf(s[j][2], s[j][3]));
            }
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1));
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1));
            mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
            const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
            const float corr_a = exp2f(m_a - mn_a), corr_b = exp2f(m_b - mn_b);
            m_a = mn_a;
            m_b = mn_b;
            float sum_a = 0.f, sum_b = 0.f;
#pragma unroll
            for (int j = 0; j < NJ; ++j) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    // (a masked score is -FLT_MAX; while a row has seen no key its maximum is that too)
                    const float pv = s[j][e] > -1e37f ? exp2f(s[j][e] - (e < 2 ? mn_a : mn_b)) : 0.f;
                    s[j][e] = pv;
                    if (e < 2) sum_a += pv;
                    else sum_b += pv;
                }
            }
            l_a = l_a * corr_a + sum_a;
            l_b = l_b * corr_b + sum_b;
#pragma unroll
            for (int nb = 0; nb < DVP / 8; ++nb) {
                o[nb][0] *= corr_a;
                o[nb][1] *= corr_a;
                o[nb][2] *= corr_b;
                o[nb][3] *= corr_b;
            }
#pragma unroll
            for (int kk = 0; kk < NKK; ++kk) {
                uint32_t pa[4];
                pa[0] = dv_pack(s[2 * kk][0], s[2 * kk][1]);
                pa[1] = dv_pack(s[2 * kk][2], s[2 * kk][3]);
                pa[2] = dv_pack(s[2 * kk + 1][0], s[2 * kk + 1][1]);
                pa[3] = dv_pack(s[2 * kk + 1][2], s[2 * kk + 1][3]);
                const uint32_t vaddr = (uint32_t)__cvta_generic_to_shared(vb + (kk * 16 + (lane & 15)) * VS);
#pragma unroll
                for (int nb = 0; nb < DVP / 8; ++nb) {
                    uint32_t b0, b1;
                    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];"
                                 : "=r"(b0), "=r"(b1) : "r"(vaddr + nb * 16));
                    dv_mma_16816(o[nb], pa, b0, b1);
                }
            }
        }
        __syncthreads();
    }
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 1);
    l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 1);
    l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
    const float lambda = a.lambda[0];
    bf16* out = (bf16*)a.out;

    if constexpr (NARROW) {
        // every warp holds the same 16 rows of its map over its own keys: they meet in shared memory
        constexpr int PS = L::PS, NC = (DVP + 31) / 32;
        float* part = reinterpret_cast<float*>(diff_smem);        // [map * 4 + sub][16][PS]
        float* mine = part + (warp * 16) * PS;
        __syncthreads();                               // (a block with no tile comes here from zeroing the padding)
#pragma unroll
        for (int nb = 0; nb < DVP / 8; ++nb) {
            *reinterpret_cast<float2*>(&mine[gid * PS + nb * 8 + 2 * tid4]) = make_float2(o[nb][0], o[nb][1]);
            *reinterpret_cast<float2*>(&mine[(gid + 8) * PS + nb * 8 + 2 * tid4]) = make_float2(o[nb][2], o[nb][3]);
        }
        if (tid4 == 0) {
            mine[gid * PS + DVP] = m_a;
            mine[gid * PS + DVP + 1] = l_a;
            mine[(gid + 8) * PS + DVP] = m_b;
            mine[(gid + 8) * PS + DVP + 1] = l_b;
        }
        __syncthreads();
        const int rows_here = last_row - tile_row0 + 1;
        for (int row_l = warp; row_l < rows_here; row_l += 8) {   // a warp brings a row together
            float y[2][NC], mm[2], den[2];
#pragma unroll
            for (int mp = 0; mp < 2; ++mp) {
                const float* src = part + ((size_t)mp * 4 * 16 + row_l) * PS;
                mm[mp] = -FLT_MAX;
                den[mp] = 0.f;
#pragma unroll
                for (int w = 0; w < 4; ++w) mm[mp] = fmaxf(mm[mp], src[w * 16 * PS + DVP]);
                float f[4];
#pragma unroll
                for (int w = 0; w < 4; ++w) {
                    f[w] = exp2f(src[w * 16 * PS + DVP] - mm[mp]);
                    den[mp] += f[w] * src[w * 16 * PS + DVP + 1];
                }
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    const int d = lane + 32 * c;
                    y[mp][c] = 0.f;
                    if (d < dv) {
#pragma unroll
                        for (int w = 0; w < 4; ++w) y[mp][c] += f[w] * src[w * 16 * PS + d];
                    }
                }
            }
            if (ksplit > 1) {                          // sums relative to mm, then mm and the weights' sum, map by map
                float* dst = scratch + (((((size_t)r * nkv + g) * (gridDim.x / ksplit) + row_tile) * ksplit + key_part) * 16 + row_l) * 2 * (dv + 2);
#pragma unroll
                for (int mp = 0; mp < 2; ++mp, dst += dv + 2) {
#pragma unroll
                    for (int c = 0; c < NC; ++c)
                        if (lane + 32 * c < dv) dst[lane + 32 * c] = y[mp][c];
                    if (lane == 0) {
                        dst[dv] = mm[mp];
                        dst[dv + 1] = den[mp];
                    }
                }
                continue;
            }
            const float i0 = den[0] > 0.f ? 1.f / den[0] : 0.f, i1 = den[1] > 0.f ? lambda / den[1] : 0.f;
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                y[0][c] = y[0][c] * i0 - y[1][c] * i1;             // (zero past dv)
                ss += y[0][c] * y[0][c];
            }
            const float mul = a.post / sqrtf(lsb_warp_sum(ss) / (float)dv + a.eps);
            const int row = tile_row0 + row_l;
            bf16* dst = out + (((size_t)qs + row / group) * nh + g * group + row % group) * dv;
#pragma unroll
            for (int c = 0; c < NC; ++c)
                if (lane + 32 * c < dv) dst[lane + 32 * c] = __float2bfloat16_rn(y[0][c] * mul);
        }
    } else {
        constexpr int YS = L::YS;
        float* ya = reinterpret_cast<float*>(diff_smem) + (sub * 16 + gid) * YS + 2 * tid4;
        float* yb = ya + 8 * YS;
        const float inv_a = l_a > 0.f ? 1.f / l_a : 0.f, inv_b = l_b > 0.f ? 1.f / l_b : 0.f;
        if (map == 1) {
#pragma unroll
            for (int nb = 0; nb < DVP / 8; ++nb) {
                *reinterpret_cast<float2*>(ya + nb * 8) = make_float2(o[nb][0] * inv_a, o[nb][1] * inv_a);
                *reinterpret_cast<float2*>(yb + nb * 8) = make_float2(o[nb][2] * inv_b, o[nb][3] * inv_b);
            }
        }
        __syncthreads();
        if (map == 1 || !active) return;
        float ss_a = 0.f, ss_b = 0.f;
#pragma unroll
        for (int nb = 0; nb < DVP / 8; ++nb) {                    // (columns past dv are zero in both maps)
            const float2 za = *reinterpret_cast<const float2*>(ya + nb * 8), zb = *reinterpret_cast<const float2*>(yb + nb * 8);
            o[nb][0] = o[nb][0] * inv_a - lambda * za.x;
            o[nb][1] = o[nb][1] * inv_a - lambda * za.y;
            o[nb][2] = o[nb][2] * inv_b - lambda * zb.x;
            o[nb][3] = o[nb][3] * inv_b - lambda * zb.y;
            ss_a += o[nb][0] * o[nb][0] + o[nb][1] * o[nb][1];
            ss_b += o[nb][2] * o[nb][2] + o[nb][3] * o[nb][3];
        }
        ss_a += __shfl_xor_sync(0xffffffffu, ss_a, 1);
        ss_a += __shfl_xor_sync(0xffffffffu, ss_a, 2);
        ss_b += __shfl_xor_sync(0xffffffffu, ss_b, 1);
        ss_b += __shfl_xor_sync(0xffffffffu, ss_b, 2);
        const float mul_a = a.post / sqrtf(ss_a / (float)dv + a.eps), mul_b = a.post / sqrtf(ss_b / (float)dv + a.eps);
#pragma unroll
        for (int nb = 0; nb < DVP / 8; ++nb) {
            if (nb < vper) {
                const int c = nb * 8 + 2 * tid4;
                if (ok_a) *reinterpret_cast<__nv_bfloat162*>(out + (t_a * nh + h_a) * dv + c) = __floats2bfloat162_rn(o[nb][0] * mul_a, o[nb][1] * mul_a);
                if (ok_b) *reinterpret_cast<__nv_bfloat162*>(out + (t_b * nh + h_b) * dv + c) = __floats2bfloat162_rn(o[nb][2] * mul_b, o[nb][3] * mul_b);
            }
        }
    }
}

// ------------------------------------------------------------------ rows that wait on memory
// Steps whose requests bring at most 16 rows each (single tokens: one row per query head of a kv head's
// group), values of up to 128.  A block owns a request, a kv head and 16 rows; its four warps walk the keys
// on their own, 16 at a time, each with a ring of its own in shared memory, so that no warp waits for
// another until the end.  A warp holds both maps: a chunk's values are read from shared memory once for
// both.  Chunks that hold cached keys only are asked for before the wait on the previous kernel (the
// step's metadata and the block table are in place by then).  The blocks that share a row tile's keys are
// one cluster: each leaves its sums in its shared memory, and after the cluster has met, each brings
// its share of the rows together.  LOW8: at most 8 rows, the lower half of every fragment is left alone.
constexpr int kDecWarps = 4, kDecKeys = 16;

template <int DKP, int DVP>
struct DecTile {
    static constexpr int STAGES = DKP == 64 ? 3 : 2;
    static constexpr int KS = 2 * DKP + 8, VS = DVP + 8;    // row strides in elements: 4 words past a multiple of 32
    static constexpr int PS = DVP + 2;                      // a row of sums: O, then m and l
    static constexpr int kStage = kDecKeys * (KS + VS);     // elements of a warp's chunk
    static constexpr size_t kRing = (size_t)kDecWarps * STAGES * kStage * 2;
    static constexpr size_t kMeet = (size_t)(kDecWarps + 1) * 16 * 2 * PS * 4;
    static constexpr size_t kTotal = kRing > kMeet ? kRing : kMeet;
};

__device__ __forceinline__ float diff_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float ld_peer(const float* p, uint32_t rank) {
    uint32_t peer;
    float v;
    asm("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(peer) : "r"((uint32_t)__cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(peer) : "memory");
    return v;
}
__device__ __forceinline__ void cluster_meet() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int DKP, int DVP, bool LOW8>
__global__ void __launch_bounds__(kDecWarps * 32, 2)
attention_diff_decode_kernel(const DiffArgs a, float scale_log2, int ksplit) {
    using L = DecTile<DKP, DVP>;
    typedef __nv_bfloat16 bf16;
    constexpr int KS = L::KS, VS = L::VS, PS = L::PS, ST = L::STAGES, NB = DVP / 8, NC = DVP / 32;
    extern __shared__ __align__(16) unsigned char diff_smem[];
    lsb_pdl_launch_dependents();
    const int nh = a.nh, nkv = a.nkv, dk = a.dk, dv = a.dv, page_size = a.page_size;
    const int r = blockIdx.z, g = blockIdx.y, group = nh / nkv;
    const int qs = a.q_start[r];
    const int q_len = a.q_start[r + 1] - qs;
    const int rows_total = q_len * group;
    const int row_tile = blockIdx.x / ksplit, part_id = blockIdx.x % ksplit;
    const int tile_row0 = row_tile * 16;
    if (tile_row0 >= rows_total) return;               // (every block of a cluster leaves here, or none)
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tid4 = lane & 3;
    const int p_base = a.kv_len[r] - q_len;
    const int rows_here = min(16, rows_total - tile_row0);
    const int last_pos = p_base + (tile_row0 + rows_here - 1) / group;
    const int first_pos = p_base + tile_row0 / group;
    const int key_lo = diff_lowest(first_pos, a.window, a.chunk);      // the first key any row of the block sees
    const int last_lo = diff_lowest(last_pos, a.window, a.chunk);
    int c0 = key_lo / kDecKeys, c1 = last_pos / kDecKeys + 1;
    {                                                  // this block's share of the chunks (it may be empty)
        const int per = (c1 - c0 + ksplit - 1) / ksplit;
        c0 += part_id * per;
        c1 = min(c1, c0 + per);
    }
    const int n = max(0, (c1 - c0 - warp + kDecWarps - 1) / kDecWarps);      // chunks c0 + warp, + 4, ...
    const int* bt = a.block_table + (size_t)a.table_rows[r] * a.table_stride;
    bf16* ring = reinterpret_cast<bf16*>(diff_smem) + warp * ST * L::kStage;
    // the padding of the rows is zeroed once; copies never touch it
    if (dk < DKP || dv < DVP) {
        for (int row = lane; row < ST * kDecKeys; row += 32) {
            bf16* kd = ring + (row / kDecKeys) * L::kStage + (row % kDecKeys) * KS;
            bf16* vd = ring + (row / kDecKeys) * L::kStage + kDecKeys * KS + (row % kDecKeys) * VS;
            for (int c = dk; c < DKP; ++c) kd[c] = kd[DKP + c] = __float2bfloat16_rn(0.f);
            for (int c = dv; c < DVP; ++c) vd[c] = __float2bfloat16_rn(0.f);
        }
        __syncwarp();
    }
    // A chunk's copies: the warp takes a key at a time, a lane 16 bytes of the key's rows (first the keys of
    // both maps, then the values).  A chunk's place is looked up a chunk ahead of the copies.  Pages of a
    // multiple of 16 keys hold a chunk whole, its rows one after the other (rows past the last key and
    // before the first are then copied too: they are finite and masked); other pages go key by key.
    constexpr int kIter = (2 * DKP / 8 + DVP / 8 + 31) / 32;
    const bool whole = page_size % kDecKeys == 0;
    const int kper = dk >> 3, nk = 2 * kper, nv = dv >> 3;
    const char* src0[kIter];                           // this lane's 16 bytes of row 0 of the pages
    int src_step[kIter], dst_step[kIter];              // bytes from row to row there, and in the ring
    uint32_t dst0[kIter];
    bool mine[kIter];
#pragma unroll
    for (int u = 0; u < kIter; ++u) {
        const int c = lane + 32 * u;
        const bool is_k = c < nk;
        mine[u] = c < nk + nv;
        src0[u] = is_k ? (const char*)a.k_pages + c * 16 : (const char*)a.v_pages + (c - nk) * 16;
        src_step[u] = (is_k ? 2 * dk : dv) * 2;
        dst0[u] = (uint32_t)__cvta_generic_to_shared(ring) +
                  2u * (uint32_t)(is_k ? (c >= kper ? DKP + (c - kper) * 8 : c * 8) : kDecKeys * KS + (c - nk) * 8);
        dst_step[u] = (is_k ? KS : VS) * 2;
    }
    constexpr int kBad = -2, kNone = -1;
    auto place = [&](int k) -> int {                   // (not looked at before the copies of a later turn)
        const int key = (c0 + warp + k * kDecWarps) * kDecKeys + (whole ? 0 : lane & 15);
        if (k >= n || (!whole && (key > last_pos || key < key_lo))) return kNone;
        const int page = bt[key / page_size];
        return page < 0 ? kBad : page;
    };
    auto issue = [&](int page, int k, int st) {
        const int key = (c0 + warp + k * kDecWarps) * kDecKeys + (whole ? 0 : lane & 15);
        long long at = -1;
        if (page >= a.num_pages || page == kBad) lsb_set_status(LSB_BAD_PAGE);
        else if (page >= 0) at = ((long long)page * nkv + g) * page_size + key % page_size;
        if (whole) {
            const int size = at >= 0 ? 16 : 0;         // (0: filled with zeros)
            const long long row = at >= 0 ? at : 0;
#pragma unroll
            for (int u = 0; u < kIter; ++u) {
                if (mine[u]) {
                    const char* src = src0[u] + row * src_step[u];
                    uint32_t dst = dst0[u] + (uint32_t)(st * L::kStage * 2);
#pragma unroll
                    for (int i = 0; i < kDecKeys; ++i) {
                        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(size) : "memory");
                        src += src_step[u];
                        dst += dst_step[u];
                    }
                }
            }
            return;
        }
#pragma unroll 1
        for (int i = 0; i < kDecKeys; ++i) {
            const long long row = __shfl_sync(0xffffffffu, at, i);
            const int size = row >= 0 ? 16 : 0;
#pragma unroll
            for (int u = 0; u < kIter; ++u)
                if (mine[u])
                    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;"
                                 ::"r"(dst0[u] + (uint32_t)(st * L::kStage * 2 + i * dst_step[u])),
                                   "l"(src0[u] + (row >= 0 ? row * src_step[u] : 0)), "r"(size) : "memory");
        }
    };
    auto commit = [] { asm volatile("cp.async.commit_group;" ::: "memory"); };
    int pages[ST - 1];
#pragma unroll
    for (int st = 0; st < ST - 1; ++st) pages[st] = place(st);
    // chunks of keys that earlier steps cached do not depend on the kernel before
    int early = 0;
#pragma unroll
    for (int st = 0; st < ST - 1; ++st)
        if (st < n && (c0 + warp + st * kDecWarps + 1) * kDecKeys <= p_base) early = st + 1;
#pragma unroll
    for (int st = 0; st < ST - 1; ++st) {
        if (st < early) {
            issue(pages[st], st, st);
            commit();
        }
    }
    int at_next = place(ST - 1);
    lsb_pdl_wait();
#pragma unroll
    for (int st = 0; st < ST - 1; ++st) {
        if (st >= early) {
            if (st < n) issue(pages[st], st, st);
            commit();
        }
    }

    // this thread's two rows (gid and gid + 8)
    const int row_a = tile_row0 + gid, row_b = row_a + 8;
    const bool ok_a = row_a < rows_total, ok_b = !LOW8 && row_b < rows_total;
    const int pos_a = p_base + row_a / group, pos_b = p_base + row_b / group;
    const int lo_a = diff_lowest(pos_a, a.window, a.chunk), lo_b = diff_lowest(pos_b, a.window, a.chunk);
    uint32_t qa[2][DKP / 16][4];
    {
        const bf16* qa_row = (const bf16*)a.q + (((size_t)qs + row_a / group) * nh + g * group + row_a % group) * (2 * dk);
        const bf16* qb_row = (const bf16*)a.q + (((size_t)qs + row_b / group) * nh + g * group + row_b % group) * (2 * dk);
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
#pragma unroll
            for (int ks = 0; ks < DKP / 16; ++ks) {
                uint32_t(&f)[4] = qa[mp][ks];
                f[0] = f[1] = f[2] = f[3] = 0u;
                const int c = mp * dk + ks * 16 + 2 * tid4;
                if (ks * 16 < dk) {
                    if (ok_a) f[0] = *reinterpret_cast<const uint32_t*>(qa_row + c);
                    if (ok_b) f[1] = *reinterpret_cast<const uint32_t*>(qb_row + c);
                }
                if (ks * 16 + 8 < dk) {
                    if (ok_a) f[2] = *reinterpret_cast<const uint32_t*>(qa_row + c + 8);
                    if (ok_b) f[3] = *reinterpret_cast<const uint32_t*>(qb_row + c + 8);
                }
            }
        }
    }
    float o[2][NB][4];
    float m_a[2], m_b[2], l_a[2], l_b[2];
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        m_a[mp] = m_b[mp] = -FLT_MAX;
        l_a[mp] = l_b[mp] = 0.f;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) o[mp][nb][0] = o[mp][nb][1] = o[mp][nb][2] = o[mp][nb][3] = 0.f;
    }
    for (int k = 0; k < n; ++k) {
        if (k + ST - 1 < n) issue(at_next, k + ST - 1, (k + ST - 1) % ST);
        commit();                                      // (a group a turn, real or not)
        at_next = place(k + ST);
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
        __syncwarp();
        const bf16* kb = ring + (k % ST) * L::kStage;
        const int key0 = (c0 + warp + k * kDecWarps) * kDecKeys;
        const bool interior = key0 >= last_lo && key0 + kDecKeys - 1 <= first_pos;
        uint32_t pa[2][4];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
            const uint32_t kaddr = (uint32_t)__cvta_generic_to_shared(kb + ((lane & 7) + (lane >> 4) * 8) * KS + mp * DKP + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int ks = 0; ks < DKP / 16; ++ks) {
                uint32_t b[4];
                asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                             : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(kaddr + ks * 32));
                dv_mma_16816(s[0], qa[mp][ks], b[0], b[1]);
                dv_mma_16816(s[1], qa[mp][ks], b[2], b[3]);
            }
            constexpr int NE = LOW8 ? 2 : 4;
#pragma unroll
            for (int j = 0; j < 2; ++j) {
#pragma unroll
                for (int e = 0; e < NE; ++e) s[j][e] *= scale_log2;
            }
            if (!interior) {
#pragma unroll
                for (int j = 0; j < 2; ++j) {
#pragma unroll
                    for (int e = 0; e < NE; ++e) {
                        const int key = key0 + j * 8 + 2 * tid4 + (e & 1);
                        if (e < 2 ? (key < lo_a || key > pos_a) : (key < lo_b || key > pos_b)) s[j][e] = -INFINITY;
                    }
                }
            }
            float mx_a = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1])), mx_b = -FLT_MAX;
            if (!LOW8) mx_b = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1));
            mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
            if (!LOW8) {
                mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1));
                mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
            }
            // accumulators are rescaled only when a maximum has moved
            if (__any_sync(0xffffffffu, mx_a > m_a[mp] || (!LOW8 && mx_b > m_b[mp]))) {
                const float mn_a = fmaxf(m_a[mp], mx_a), corr_a = diff_exp2(m_a[mp] - mn_a);
                m_a[mp] = mn_a;
                l_a[mp] *= corr_a;
#pragma unroll
                for (int nb = 0; nb < NB; ++nb) {
                    o[mp][nb][0] *= corr_a;
                    o[mp][nb][1] *= corr_a;
                }
                if (!LOW8) {
                    const float mn_b = fmaxf(m_b[mp], mx_b), corr_b = diff_exp2(m_b[mp] - mn_b);
                    m_b[mp] = mn_b;
                    l_b[mp] *= corr_b;
#pragma unroll
                    for (int nb = 0; nb < NB; ++nb) {
                        o[mp][nb][2] *= corr_b;
                        o[mp][nb][3] *= corr_b;
                    }
                }
            }
#pragma unroll
            for (int j = 0; j < 2; ++j) {
#pragma unroll
                for (int e = 0; e < NE; ++e) {
                    // (a masked score is -inf and no maximum ever is: its weight is 0)
                    const float pv = diff_exp2(s[j][e] - (e < 2 ? m_a[mp] : m_b[mp]));
                    s[j][e] = pv;
                    if (e < 2) l_a[mp] += pv;
                    else l_b[mp] += pv;
                }
                pa[mp][2 * j] = dv_pack(s[j][0], s[j][1]);
                pa[mp][2 * j + 1] = LOW8 ? 0u : dv_pack(s[j][2], s[j][3]);
            }
        }
        const uint32_t vaddr = (uint32_t)__cvta_generic_to_shared(kb + kDecKeys * KS + (lane & 15) * VS + (lane >> 4) * 8);
#pragma unroll
        for (int nb = 0; nb < NB; nb += 2) {
            uint32_t b[4];
            asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                         : "=r"(b[0]), "=r"(b[1]), "=r"(b[2]), "=r"(b[3]) : "r"(vaddr + nb * 16));
#pragma unroll
            for (int mp = 0; mp < 2; ++mp) {
                dv_mma_16816(o[mp][nb], pa[mp], b[0], b[1]);
                dv_mma_16816(o[mp][nb + 1], pa[mp], b[2], b[3]);
            }
        }
        __syncwarp();                                  // the chunk's buffer may be filled again
    }
    asm volatile("cp.async.wait_all;" ::: "memory");
    __syncthreads();
    // the four warps' sums meet in shared memory
    float* part = reinterpret_cast<float*>(diff_smem);       // [warp][row][map][PS]
    float* comb = part + kDecWarps * 16 * 2 * PS;            // [row][map][PS]: the block's sums, for its cluster
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        l_a[mp] += __shfl_xor_sync(0xffffffffu, l_a[mp], 1);
        l_a[mp] += __shfl_xor_sync(0xffffffffu, l_a[mp], 2);
        float* da = part + ((warp * 16 + gid) * 2 + mp) * PS;
#pragma unroll
        for (int nb = 0; nb < NB; ++nb) *reinterpret_cast<float2*>(&da[nb * 8 + 2 * tid4]) = make_float2(o[mp][nb][0], o[mp][nb][1]);
        if (tid4 == 0) {
            da[DVP] = m_a[mp];
            da[DVP + 1] = l_a[mp];
        }
        if (!LOW8) {
            l_b[mp] += __shfl_xor_sync(0xffffffffu, l_b[mp], 1);
            l_b[mp] += __shfl_xor_sync(0xffffffffu, l_b[mp], 2);
            float* db = da + 8 * 2 * PS;
#pragma unroll
            for (int nb = 0; nb < NB; ++nb) *reinterpret_cast<float2*>(&db[nb * 8 + 2 * tid4]) = make_float2(o[mp][nb][2], o[mp][nb][3]);
            if (tid4 == 0) {
                db[DVP] = m_b[mp];
                db[DVP + 1] = l_b[mp];
            }
        }
    }
    __syncthreads();
    const float lambda = a.lambda[0];
    auto finish = [&](float (&y)[2][NC], const float (&den)[2], int row_l) {
        const float i0 = den[0] > 0.f ? 1.f / den[0] : 0.f, i1 = den[1] > 0.f ? lambda / den[1] : 0.f;
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            y[0][c] = y[0][c] * i0 - y[1][c] * i1;           // (zero past dv)
            ss += y[0][c] * y[0][c];
        }
        const float mul = a.post / sqrtf(lsb_warp_sum(ss) / (float)dv + a.eps);
        const int row = tile_row0 + row_l;
        bf16* dst = (bf16*)a.out + (((size_t)qs + row / group) * nh + g * group + row % group) * dv;
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (lane + 32 * c < dv) dst[lane + 32 * c] = __float2bfloat16_rn(y[0][c] * mul);
    };
    for (int row_l = warp; row_l < rows_here; row_l += kDecWarps) {      // a warp brings a row together
        float y[2][NC], den[2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            const float* src = part + (row_l * 2 + mp) * PS;
            constexpr int WS = 16 * 2 * PS;
            float mm = -FLT_MAX, f[kDecWarps];
            den[mp] = 0.f;
#pragma unroll
            for (int w = 0; w < kDecWarps; ++w) mm = fmaxf(mm, src[w * WS + DVP]);
#pragma unroll
            for (int w = 0; w < kDecWarps; ++w) {
                f[w] = exp2f(src[w * WS + DVP] - mm);
                den[mp] += f[w] * src[w * WS + DVP + 1];
            }
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                y[mp][c] = 0.f;
#pragma unroll
                for (int w = 0; w < kDecWarps; ++w) y[mp][c] += f[w] * src[w * WS + lane + 32 * c];
            }
            if (ksplit > 1) {
                float* dst = comb + (row_l * 2 + mp) * PS;
#pragma unroll
                for (int c = 0; c < NC; ++c) dst[lane + 32 * c] = y[mp][c];
                if (lane == 0) {
                    dst[DVP] = mm;
                    dst[DVP + 1] = den[mp];
                }
            }
        }
        if (ksplit == 1) finish(y, den, row_l);
    }
    if (ksplit == 1) return;
    cluster_meet();
    for (int row_l = part_id * kDecWarps + warp; row_l < rows_here; row_l += ksplit * kDecWarps) {
        float y[2][NC], den[2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            const float* src = comb + (row_l * 2 + mp) * PS;
            float f[kMaxParts], l[kMaxParts], v[kMaxParts][NC], mm = -FLT_MAX;
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {            // all peers' values in flight at once
                f[p] = p < ksplit ? ld_peer(src + DVP, p) : -FLT_MAX;
                l[p] = p < ksplit ? ld_peer(src + DVP + 1, p) : 0.f;
#pragma unroll
                for (int c = 0; c < NC; ++c) v[p][c] = p < ksplit ? ld_peer(src + lane + 32 * c, p) : 0.f;
            }
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) mm = fmaxf(mm, f[p]);
            den[mp] = 0.f;
#pragma unroll
            for (int c = 0; c < NC; ++c) y[mp][c] = 0.f;
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {            // summed in rank order
                const float w = p < ksplit ? exp2f(f[p] - mm) : 0.f;
                den[mp] += w * l[p];
#pragma unroll
                for (int c = 0; c < NC; ++c) y[mp][c] += w * v[p][c];
            }
        }
        finish(y, den, row_l);
    }
    cluster_meet();                                    // nobody leaves while a peer may still read its shared memory
}

// The partial sums of `ksplit` blocks that shared a row tile's keys, brought together, differenced and
// normed: scratch [request, kv head, row tile, part, 16 rows, map, dv + 2].  A warp owns a row.
template <int NC>
__global__ void __launch_bounds__(kDiffThreads)
attention_diff_merge_kernel(const float* __restrict__ scratch, const DiffArgs a, int ksplit) {
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int r = blockIdx.z, g = blockIdx.y, group = a.nh / a.nkv, dv = a.dv;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int qs = a.q_start[r];
    const int rows_total = (a.q_start[r + 1] - qs) * group;
    const int tile_row0 = blockIdx.x * 16;
    if (tile_row0 >= rows_total) return;
    const int rows_here = min(16, rows_total - tile_row0);
    const float* base = scratch + (((size_t)r * a.nkv + g) * gridDim.x + blockIdx.x) * ksplit * 16 * 2 * (dv + 2);
    const float lambda = a.lambda[0];
    for (int row_l = warp; row_l < rows_here; row_l += 8) {
        float y[2][NC], inv[2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            float f[kMaxParts], l[kMaxParts], mm = -FLT_MAX, den = 0.f;
            const float* src[kMaxParts];
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {
                src[p] = base + (((size_t)(p < ksplit ? p : 0) * 16 + row_l) * 2 + mp) * (dv + 2);
                f[p] = p < ksplit ? src[p][dv] : -FLT_MAX;
                l[p] = p < ksplit ? src[p][dv + 1] : 0.f;
            }
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) mm = fmaxf(mm, f[p]);
#pragma unroll
            for (int p = 0; p < kMaxParts; ++p) {
                f[p] = p < ksplit ? exp2f(f[p] - mm) : 0.f;
                den += f[p] * l[p];
            }
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                y[mp][c] = 0.f;
                if (lane + 32 * c < dv) {
#pragma unroll
                    for (int p = 0; p < kMaxParts; ++p) y[mp][c] += p < ksplit ? f[p] * src[p][lane + 32 * c] : 0.f;
                }
            }
            inv[mp] = den > 0.f ? 1.f / den : 0.f;
        }
        float ss = 0.f;
#pragma unroll
        for (int c = 0; c < NC; ++c) {
            y[0][c] = y[0][c] * inv[0] - lambda * (y[1][c] * inv[1]);
            ss += y[0][c] * y[0][c];
        }
        const float mul = a.post / sqrtf(lsb_warp_sum(ss) / (float)dv + a.eps);
        const int row = tile_row0 + row_l;
        __nv_bfloat16* dst = (__nv_bfloat16*)a.out + (((size_t)qs + row / group) * a.nh + g * group + row % group) * dv;
#pragma unroll
        for (int c = 0; c < NC; ++c)
            if (lane + 32 * c < dv) dst[lane + 32 * c] = __float2bfloat16_rn(y[0][c] * mul);
    }
}

// ------------------------------------------------------------------ host side
// How a step of this shape is launched, as dv_mma_plan says (16-row blocks or not, tiles in flight, blocks that
// share a row tile's keys); bit 2: the kernel whose warps walk the keys on their own, for steps of at
// most 16 rows a request and values of up to 128.  shape 5 and more: that kernel with keys shared by
// shape - 4 blocks; 1 - 4 as in dv_mma_plan.
static int diff_plan(int n_requests, int max_q_len, int nh, int nkv, int dv, int chunk, int sms, int shape) {
    const long long rows = (long long)max_q_len * (nh / nkv);
    if (dv > 128 || (shape == 0 && rows > 16) || (shape >= 1 && shape <= 4))
        return dv_mma_plan(n_requests, max_q_len, nh, nkv, chunk, sms, shape > 4 ? 0 : shape);
    if (sms <= 0) sms = 148;
    const long long thin = (rows + 15) / 16 * nkv * n_requests;
    long long ksplit = shape > 4 ? shape - 4 : (2 * sms) / thin;       // two blocks fit an SM
    if (ksplit > kMaxParts) ksplit = kMaxParts;
    if (shape == 0 && chunk > 0 && ksplit > (chunk + kMmaKeys - 1) / kMmaKeys) ksplit = (chunk + kMmaKeys - 1) / kMmaKeys;
    if (ksplit < 1) ksplit = 1;
    return 4 | ((int)ksplit << 8);
}
LSB_API int lsb_attention_diff_plan(int n_requests, int max_q_len, int nh, int nkv, int dv, int chunk, int sms, int shape) {
    return diff_plan(n_requests, max_q_len, nh, nkv, dv, chunk, sms, shape);
}

LSB_API int lsb_attention_diff_mma_supported(int dk, int dv) {
    return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 128 && dv <= 256;
}

LSB_API int lsb_attention_diff_max_dim() { return kDiffMaxDim; }

static DiffArgs diff_args(const void* q, const void* k_pages, const void* v_pages, const int* q_start, const int* kv_len,
                          const int* table_rows, const int* block_table, int table_stride, void* out, int nh, int nkv,
                          int dk, int dv, int page_size, int num_pages, float scale, int window, int chunk,
                          const float* lambda, float eps, float post) {
    DiffArgs a;
    a.q = q; a.k_pages = k_pages; a.v_pages = v_pages;
    a.q_start = q_start; a.kv_len = kv_len; a.table_rows = table_rows; a.block_table = block_table;
    a.table_stride = table_stride; a.out = out;
    a.nh = nh; a.nkv = nkv; a.dk = dk; a.dv = dv; a.page_size = page_size; a.num_pages = num_pages;
    a.scale = scale; a.window = window; a.chunk = chunk; a.lambda = lambda; a.eps = eps; a.post = post;
    return a;
}

template <int DKP, int DVP, int STAGES, bool NARROW>
static int launch_mma(const DiffArgs& a, dim3 grid, int ksplit, float* scratch, cudaStream_t stream) {
    constexpr size_t smem = DiffTile<DKP, DVP, STAGES, NARROW>::kTotal;
    if (smem > 48 * 1024) {
        const int rc = (int)cudaFuncSetAttribute(attention_diff_mma_kernel<DKP, DVP, STAGES, NARROW>,
                                                 cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (rc) return rc;
    }
    return lsb_launch(attention_diff_mma_kernel<DKP, DVP, STAGES, NARROW>, grid, dim3(kDiffThreads), smem, stream, 1, a,
                      a.scale * 1.4426950408889634f, ksplit, scratch);
}

template <int DKP, int DVP>
static int launch_shape(const DiffArgs& a, int plan, dim3 grid, float* scratch, cudaStream_t stream) {
    constexpr int kDeep = DiffTile<DKP, DVP, 4, true>::kTotal <= 220 * 1024 ? 4 : 3;
    const int ksplit = plan >> 8;
    if (!(plan & 1)) return launch_mma<DKP, DVP, 2, false>(a, grid, 1, scratch, stream);
    return plan & 2 ? launch_mma<DKP, DVP, kDeep, true>(a, grid, ksplit, scratch, stream)
                    : launch_mma<DKP, DVP, 2, true>(a, grid, ksplit, scratch, stream);
}

template <int DKP, int DVP, bool LOW8>
static int launch_decode_rows(const DiffArgs& a, dim3 grid, int ksplit, cudaStream_t stream) {
    constexpr size_t smem = DecTile<DKP, DVP>::kTotal;
    static_assert(2 * (smem + 1024) <= 228 * 1024, "two blocks an SM");
    static int configured = -1;
    if (configured < 0)
        configured = (int)cudaFuncSetAttribute(attention_diff_decode_kernel<DKP, DVP, LOW8>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (configured) return configured;
    return lsb_launch(attention_diff_decode_kernel<DKP, DVP, LOW8>, grid, dim3(kDecWarps * 32), smem, stream, ksplit, a,
                      a.scale * 1.4426950408889634f, ksplit);
}

template <int DKP, int DVP>
static int launch_decode(const DiffArgs& a, dim3 grid, int ksplit, bool low8, cudaStream_t stream) {
    return low8 ? launch_decode_rows<DKP, DVP, true>(a, grid, ksplit, stream) : launch_decode_rows<DKP, DVP, false>(a, grid, ksplit, stream);
}

// bfloat16; q, the pages and out 16-byte aligned; sms: the device's multiprocessors (what a small grid is
// measured against); scratch: n_requests * nkv * row tiles * parts * 16 * 2 * (dv + 2) floats if the plan has parts.
LSB_API int lsb_attention_diff_mma(const void* q, const void* k_pages, const void* v_pages, const int* q_start,
                                   const int* kv_len, const int* table_rows, const int* block_table, int table_stride,
                                   void* out, int n_requests, int max_q_len, int nh, int nkv, int dk, int dv, int page_size,
                                   int num_pages, float scale, int window, int chunk, const float* lambda, float eps,
                                   float post, int sms, int shape, float* scratch, cudaStream_t stream) {
    if (n_requests <= 0 || max_q_len <= 0) return 0;
    if (!lsb_attention_diff_mma_supported(dk, dv) || nkv <= 0 || nh % nkv || window < 0 || chunk < 0 || n_requests > 65535 ||
        nkv > 65535 || !lambda || page_size <= 0)
        return (int)cudaErrorInvalidValue;
    const DiffArgs a = diff_args(q, k_pages, v_pages, q_start, kv_len, table_rows, block_table, table_stride, out, nh, nkv,
                                 dk, dv, page_size, num_pages, scale, window, chunk, lambda, eps, post);
    const long long rows = (long long)max_q_len * (nh / nkv);
    const int plan = diff_plan(n_requests, max_q_len, nh, nkv, dv, chunk, sms, shape);
    if (plan & 4) {
        const dim3 dgrid((unsigned)((rows + 15) / 16) * (plan >> 8), nkv, n_requests);
        if (dk <= 64) return dv <= 64 ? launch_decode<64, 64>(a, dgrid, plan >> 8, rows <= 8, stream) : launch_decode<64, 128>(a, dgrid, plan >> 8, rows <= 8, stream);
        return dv <= 64 ? launch_decode<128, 64>(a, dgrid, plan >> 8, rows <= 8, stream) : launch_decode<128, 128>(a, dgrid, plan >> 8, rows <= 8, stream);
    }
    const int ksplit = plan >> 8;
    if (ksplit > 1 && !scratch) return (int)cudaErrorInvalidValue;
    const unsigned tiles = (unsigned)(plan & 1 ? (rows + 15) / 16 : (rows + kMmaRows - 1) / kMmaRows);
    dim3 grid(tiles * ksplit, nkv, n_requests);
    int rc;
#define LSB_DIFF_V(DKP)                                                                       \
    (dv <= 64 ? launch_shape<DKP, 64>(a, plan, grid, scratch, stream)                         \
              : dv <= 128 ? launch_shape<DKP, 128>(a, plan, grid, scratch, stream)            \
                          : launch_shape<DKP, 256>(a, plan, grid, scratch, stream))
    rc = dk <= 64 ? LSB_DIFF_V(64) : LSB_DIFF_V(128);
#undef LSB_DIFF_V
    if (rc || ksplit <= 1) return rc;
    const dim3 mgrid(tiles, nkv, n_requests);
    if (dv <= 64) return lsb_launch(attention_diff_merge_kernel<2>, mgrid, dim3(kDiffThreads), 0, stream, 1, (const float*)scratch, a, ksplit);
    if (dv <= 128) return lsb_launch(attention_diff_merge_kernel<4>, mgrid, dim3(kDiffThreads), 0, stream, 1, (const float*)scratch, a, ksplit);
    return lsb_launch(attention_diff_merge_kernel<8>, mgrid, dim3(kDiffThreads), 0, stream, 1, (const float*)scratch, a, ksplit);
}

LSB_API int lsb_attention_diff_generic(const void* q, const void* k_pages, const void* v_pages, const int* q_start,
                                       const int* kv_len, const int* table_rows, const int* block_table, int table_stride,
                                       void* out, int dtype, int n_requests, int max_q_len, int nh, int nkv, int dk, int dv,
                                       int page_size, int num_pages, float scale, int window, int chunk, const float* lambda,
                                       float eps, float post, cudaStream_t stream) {
    if (n_requests <= 0 || max_q_len <= 0) return 0;
    if (dk <= 0 || 2 * dk > kDiffMaxDim || dv <= 0 || dv > kDiffMaxDim || nkv <= 0 || nh % nkv || window < 0 || chunk < 0 ||
        !lambda || page_size <= 0 || n_requests > 65535 || nh > 65535)
        return (int)cudaErrorInvalidValue;
    const DiffArgs a = diff_args(q, k_pages, v_pages, q_start, kv_len, table_rows, block_table, table_stride, out, nh, nkv,
                                 dk, dv, page_size, num_pages, scale, window, chunk, lambda, eps, post);
    const int al = dtype == LSB_F32 ? 4 : 8;
    const int vec = (dk % al == 0 && (uintptr_t)k_pages % 16 == 0) ? 1 : 0;
    dim3 grid((max_q_len + kDiffWarps - 1) / kDiffWarps, nh, n_requests);
    LSB_DISPATCH_DTYPE(dtype, return lsb_launch(attention_diff_generic_kernel<T>, grid, dim3(kDiffWarps * 32), 0, stream, 1, a, vec));
    return 0;
}
