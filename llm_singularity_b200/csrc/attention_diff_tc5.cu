// Differential attention of prompt portions on the 5th-generation tensor cores (bfloat16; keys of a map up
// to 128, values up to 128, both multiples of 8).  What is computed is as in attention_diff.cu.
//
// One thread block per (128-query tile, head, request), both maps side by side on the same tiles of 64
// keys: a tile's keys (both maps) and values come once by TMA, page by page through the block table, and
// serve two pipelines that otherwise know nothing of one another.  Each pipeline is that of
// attention_tc5.cu: S = Q K^T into tensor memory, four softmax warps with a query row per thread, P back
// into tensor memory as the A operand of O += P V, O rescaled only when a row's maximum has outgrown its
// reference by 2^8.  Two S buffers a map; P of a tile takes the place of that tile's S (it is in
// registers by then), so S of tile t + 2 is issued once the P V product of tile t has landed.  Tensor
// memory: 2 x (2 x 64 + values) columns, all 512 of it for values of 128.
// At the end the eight softmax warps meet once to exchange their rows' sums and then each map's warps
// take half of the value columns of both accumulators: the difference, its mean of squares (the halves
// exchanged), the norm, the store.
// Boxes are 64 wide whatever the sizes: what lies past a map's keys or the values is filled with zeros
// by the copy.  Warps: 0 TMA, 1 and 2 issue S of map 0 and 1, 3 and 12 issue P V, 4-7 and 8-11 softmax.
#include "common.cuh"

#include <cuda.h>

LSB_DEFINE_STATUS()

#include "attention_tc5.cuh"

constexpr int kThreads = 416;
constexpr int kBtCache = 512;         // block-table entries of this block's key range kept in smem

struct DiffTcParams {
    const int* q_start;
    const int* kv_len;
    const int* table_rows;
    const int* block_table;
    int table_stride;
    bf16* out;
    int nh, nkv, dv, page_size, page_shift, num_pages;
    float scale;
    int window;
    const float* lambda;
    float eps, post;
};

template <int D, int V>
struct DiffSmem {
    static constexpr int kKB = D / 64, kVB = V / 64;        // 64-wide blocks of a map's keys and of the values
    static constexpr int kStages = D == 64 ? 5 : 3;
    static constexpr int kQBytes = 2 * kRows * D * 2;
    static constexpr int kKBytes = 2 * kKeys * D * 2, kVBytes = kKeys * V * 2;
    static constexpr int kStageBytes = kKBytes + kVBytes;
    static constexpr size_t kTotal = 1024 + kQBytes + (size_t)kStages * kStageBytes + kBtCache * 4 + 4 * kRows * 4 + 40 * 8;
};

template <int D, int V>
__global__ void __launch_bounds__(kThreads, 1)
prefill_attention_diff_tc5_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                                  const __grid_constant__ CUtensorMap map_v, const DiffTcParams prm) {
    using L = DiffSmem<D, V>;
    constexpr int KB = L::kKB, VB = L::kVB, ST = L::kStages;
    constexpr uint32_t kMapCols = 2 * kKeys + V, kTmemCols = 512;
    static_assert(2 * kMapCols <= 512, "both maps' scores and accumulators live in tensor memory");
    extern __shared__ unsigned char smem_raw[];
    unsigned char* base = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned char* sQ = base;                                // [map][KB][128 rows][128 B]
    unsigned char* sKV = sQ + L::kQBytes;                    // [stages]: [map][KB][64 keys][128 B], [VB][64 keys][128 B]
    int* sBT = reinterpret_cast<int*>(sKV + ST * L::kStageBytes);
    float* sL = reinterpret_cast<float*>(sBT + kBtCache);    // [map][128]: 1 / sum of a row's weights
    float* sSS = sL + 2 * kRows;                             // [half][128]: sums of squares
    uint64_t* bars = reinterpret_cast<uint64_t*>(sSS + 2 * kRows);
    uint64_t* q_full = bars;                                 // TMA -> MMA
    uint64_t* kv_full = bars + 1;                            // [stages] TMA -> MMA
    uint64_t* kv_empty = kv_full + ST;                       // [stages] MMA -> TMA (an arrival a map)
    uint64_t* s_full = kv_empty + ST;                        // [map][2] MMA -> softmax: S of an even / odd tile
    uint64_t* p_full = s_full + 4;                           // [map][2] softmax -> MMA (an arrival a warp)
    uint64_t* o_full = p_full + 4;                           // [map][2] MMA -> softmax, S issuer: P V of an even / odd tile landed
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 4);
    __shared__ int abort_flag;

    // What follows up to the wait needs nothing from the kernel before: the step's metadata is on
    // the device before the step's first kernel starts; barriers and tensor memory are this block's.
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, r = blockIdx.z;
    const int qs = prm.q_start[r];
    const int q_len = prm.q_start[r + 1] - qs;
    const int n_qt = (q_len + kRows - 1) / kRows;
    if ((int)blockIdx.y >= n_qt) return;                     // before any barrier
    const int i0 = (n_qt - 1 - (int)blockIdx.y) * kRows;     // heavy tiles first
    const int g = h / (prm.nh / prm.nkv);
    const int kv_len = prm.kv_len[r];
    const int p0 = kv_len - q_len + i0;
    const int rows = min(kRows, q_len - i0);
    const int p_last = p0 + rows - 1;
    const int lo_cta = (prm.window > 0 && p0 - prm.window + 1 > 0) ? p0 - prm.window + 1 : 0;
    const int t0 = lo_cta / kKeys, t1 = p_last / kKeys + 1;
    const int* bt = prm.block_table + (size_t)prm.table_rows[r] * prm.table_stride;
    const int pages_per_tile = kKeys >> prm.page_shift;
    const int page_first = (t0 * kKeys) >> prm.page_shift;
    const int page_last = p_last >> prm.page_shift;          // last page that holds a needed key
    const int n_pages_here = page_last - page_first + 1;

    if (threadIdx.x == 0) {
        abort_flag = 0;
        mbar_init(q_full, 1);
        for (int s = 0; s < ST; ++s) { mbar_init(&kv_full[s], 1); mbar_init(&kv_empty[s], 2); }
        for (int i = 0; i < 4; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 4); mbar_init(&o_full[i], 1); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == 1) tmem_alloc(tmem_slot, kTmemCols);
    lsb_pdl_wait();
    // this block's slice of the block table; pages that lie wholly before the first key any row of this
    // block may see may have been given back already: their keys are masked, any page stands in for them
    const int page_needed = lo_cta >> prm.page_shift;
    for (int idx = threadIdx.x; idx < min(n_pages_here, kBtCache); idx += kThreads) {
        int page = (page_first + idx < prm.table_stride) ? bt[page_first + idx] : -1;
        if (page < 0 || page >= prm.num_pages) {
            if (page_first + idx >= page_needed) lsb_set_status(LSB_BAD_PAGE);
            page = 0;
        }
        sBT[idx] = page;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    // (only now: a block of the next kernel that took tensor memory on this SM before this one has all of its
    // own would wait for this grid's end, and this block for it)
    lsb_pdl_launch_dependents();
    const uint32_t tmem = *tmem_slot;                        // per map: S / P of even tiles, of odd tiles, O
    const int n_tiles = t1 - t0;

    if (warp == 0) {
        // ---------------------------------------------------------------- TMA producer
        if (lane == 0) {
            asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
            asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
            asm volatile("prefetch.tensormap [%0];" ::"l"(&map_v) : "memory");
            mbar_expect_tx(q_full, L::kQBytes);
            for (int m = 0; m < 2; ++m)
                for (int kb = 0; kb < KB; ++kb)
                    tma_load_3d(sQ + (m * KB + kb) * (kRows * 128), &map_q, q_full, kb * 64, 2 * h + m, qs + i0);
        }
        bool ok = true;
        for (int t = 0; t < n_tiles && ok; ++t) {
            const int s = t % ST;
            if (t >= ST) {
                if (lane == 0) ok = mbar_wait(&kv_empty[s], (uint32_t)((t / ST) - 1) & 1, &abort_flag);
                ok = __shfl_sync(0xffffffffu, ok ? 1 : 0, 0) != 0;
                if (!ok) break;
            }
            if (lane == 0) mbar_expect_tx(&kv_full[s], L::kStageBytes);
            __syncwarp();
            if (lane < pages_per_tile) {
                // pages past the last needed one repeat it: their keys are masked, their bytes finite
                int pi = (((t0 + t) * kKeys) >> prm.page_shift) + lane;
                if (pi > page_last) pi = page_last;
                const int idx = pi - page_first;
                int page;
                if (idx < kBtCache) page = sBT[idx];
                else {
                    page = pi < prm.table_stride ? bt[pi] : -1;
                    if (page < 0 || page >= prm.num_pages) {
                        if (pi >= page_needed) lsb_set_status(LSB_BAD_PAGE);
                        page = 0;
                    }
                }
                unsigned char* dst = sKV + s * L::kStageBytes + lane * prm.page_size * 128;    // (within a 64-wide block)
                for (int m = 0; m < 2; ++m)
                    for (int kb = 0; kb < KB; ++kb)
                        tma_load_5d(dst + (m * KB + kb) * (kKeys * 128), &map_k, &kv_full[s], kb * 64, m, 0, g, page);
                for (int vb = 0; vb < VB; ++vb)
                    tma_load_4d(dst + L::kKBytes + vb * (kKeys * 128), &map_v, &kv_full[s], vb * 64, 0, g, page);
            }
        }
        // copies in flight must land before the block may exit
        if (lane == 0) {
            int dummy = 0;
            mbar_wait(q_full, 0, &dummy);
            for (int t = max(0, n_tiles - ST); t < n_tiles; ++t)
                mbar_wait(&kv_full[t % ST], (uint32_t)(t / ST) & 1, &dummy);
        }
    } else if (warp == 1 || warp == 2) {
        // ---------------------------------------------------------------- MMA issuer for S of a map
        if (lane == 0) {
            const int m = warp - 1;
            constexpr uint32_t idesc_qk = make_idesc(kKeys, 0);
            uint64_t da_q[KB], db_k0[KB];
#pragma unroll
            for (int kb = 0; kb < KB; ++kb) {
                da_q[kb] = desc_kmajor(sQ + (m * KB + kb) * (kRows * 128));
                db_k0[kb] = desc_kmajor(sKV + (m * KB + kb) * (kKeys * 128));
            }
            const uint32_t ts = tmem + (uint32_t)m * kMapCols;
            bool ok = mbar_wait(q_full, 0, &abort_flag);
            for (int t = 0; t < n_tiles && ok; ++t) {
                ok = mbar_wait(&kv_full[t % ST], (uint32_t)(t / ST) & 1, &abort_flag);
                if (!ok) break;
                if (t >= 2) {                                  // P of tile t - 2 lies where this S goes
                    ok = mbar_wait(&o_full[2 * m + (t & 1)], (uint32_t)((t >> 1) - 1) & 1, &abort_flag);
                    if (!ok) break;
                }
                tc_fence_after();
                const uint64_t stage = (uint64_t)((t % ST) * (L::kStageBytes >> 4));      // address field: bytes / 16
#pragma unroll
                for (int kb = 0; kb < KB; ++kb) {
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        umma_bf16(ts + (uint32_t)((t & 1) * kKeys), da_q[kb] + 2 * k, db_k0[kb] + stage + 2 * k, idesc_qk,
                                  (kb | k) ? 1u : 0u);
                }
                umma_commit(&s_full[2 * m + (t & 1)]);
            }
        }
    } else if (warp == 3 || warp == 12) {
        // ---------------------------------------------------------------- MMA issuer for O += P V of a map
        if (lane == 0) {
            const int m = warp == 3 ? 0 : 1;
            constexpr uint32_t idesc_pv = make_idesc(V, 1);
            const uint64_t db_v0 = desc_mnmajor(sKV + L::kKBytes, kKeys * 128);
            const uint32_t ts = tmem + (uint32_t)m * kMapCols, to = ts + 2 * kKeys;
            bool ok = true;
            for (int t = 0; t < n_tiles && ok; ++t) {
                const int s = t % ST;
                // P of this tile (and O rescaled where a row's reference maximum moved)
                ok = mbar_wait(&p_full[2 * m + (t & 1)], (uint32_t)(t >> 1) & 1, &abort_flag);
                if (!ok) break;
                tc_fence_after();
                const uint64_t db = db_v0 + (uint64_t)(s * (L::kStageBytes >> 4));
                const uint32_t pa = ts + (uint32_t)((t & 1) * kKeys);
#pragma unroll
                for (int j = 0; j < kKeys / 16; ++j)           // 16 keys per MMA: eight columns of P, 16 rows of V
                    umma_bf16_ts(to, pa + j * 8, db + (uint64_t)(j * ((16 * 128) >> 4)), idesc_pv, (t | j) ? 1u : 0u);
                umma_commit(&o_full[2 * m + (t & 1)]);
                // K of this stage was read by the S product that this P descends from
                umma_commit(&kv_empty[s]);
            }
        }
    } else {
        // ---------------------------------------------------------------- softmax, one row of a map per thread
        const int m_ = (warp - 4) >> 2, q = warp & 3;
        const int il = q * 32 + lane;
        const int pos = p0 + il;
        const bool live = il < rows;
        const uint32_t lane_sel = (uint32_t)(q * 32) << 16;
        const uint32_t ts = tmem + (uint32_t)m_ * kMapCols + lane_sel, to = ts + 2 * kKeys;
        uint64_t *sf = s_full + 2 * m_, *pf = p_full + 2 * m_, *of = o_full + 2 * m_;
        const float sc = prm.scale * kLog2e;
        constexpr float kRescale = 8.f;
        float m = -INFINITY, l = 0.f;
        bool ok = true;
        uint32_t v[kKeys];
        bool loaded = false;                                   // S of tile t is on its way to v already
        for (int t = 0; t < n_tiles && ok; ++t) {
            if (!loaded) {
                ok = warp_wait(&sf[t & 1], (uint32_t)(t >> 1) & 1, &abort_flag, lane);
                if (!ok) break;
#pragma unroll
                for (int c0 = 0; c0 < kKeys; c0 += 32)
                    tmem_ld_32x32(ts + (uint32_t)((t & 1) * kKeys + c0), *reinterpret_cast<uint32_t(*)[32]>(&v[c0]));
            }
            const int key0 = (t0 + t) * kKeys;
            const bool full = key0 + kKeys - 1 <= p0 && rows == kRows && (prm.window <= 0 || key0 > p_last - prm.window);
            tmem_ld_wait();
            // columns of this tile the row may see: [c_lo, c_hi]
            const int c_hi = full ? kKeys - 1 : (live ? pos - key0 : -1);
            const int c_lo = (full || prm.window <= 0) ? 0 : pos - prm.window + 1 - key0;
            float mxa[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
            if (full) {
#pragma unroll
                for (int x = 0; x < kKeys; x += 2)
                    mxa[(x >> 1) & 3] = max3(mxa[(x >> 1) & 3], __uint_as_float(v[x]), __uint_as_float(v[x + 1]));
            } else {
#pragma unroll
                for (int x = 0; x < kKeys; ++x) {
                    const float sv = (x <= c_hi && x >= c_lo) ? __uint_as_float(v[x]) : -INFINITY;
                    v[x] = __float_as_uint(sv);
                    mxa[x & 3] = fmaxf(mxa[x & 3], sv);
                }
            }
            const float mx = fmaxf(fmaxf(mxa[0], mxa[1]), fmaxf(mxa[2], mxa[3])) * sc;      // sc > 0
            // move the reference only when needed
            float corr = 1.f;
            bool moved = false;
            if (mx > m + kRescale || (m == -INFINITY && mx > -INFINITY)) {
                corr = (m == -INFINITY) ? 0.f : fast_exp2(m - mx);
                moved = m != -INFINITY;                        // nothing accumulated before: nothing to scale
                m = mx;
                l *= corr;
            }
            const float mref = (m == -INFINITY) ? 0.f : m;
            if (t > 0 && __any_sync(0xffffffffu, moved)) {
                // O *= corr for this warp's 32 rows; the P V of the previous tile must have landed
                ok = warp_wait(&of[(t - 1) & 1], (uint32_t)((t - 1) >> 1) & 1, &abort_flag, lane);
                if (!ok) break;
#pragma unroll 1
                for (int c0 = 0; c0 < V; c0 += 32) {
                    uint32_t ov[32];
                    tmem_ld_32x32(to + c0, ov);
                    tmem_ld_wait();
#pragma unroll
                    for (int x = 0; x < 32; ++x) ov[x] = __float_as_uint(__uint_as_float(ov[x]) * corr);
                    tmem_st_32x32(to + c0, ov);
                }
                tmem_st_wait();
            }
            uint32_t s_next = 0;                               // asked early, looked at late (see attention_tc5.cu)
            if (t + 1 < n_tiles && lane == 0) s_next = mbar_test(&sf[(t + 1) & 1], (uint32_t)((t + 1) >> 1) & 1);
            // probabilities (masked scores are -inf: 2^-inf = 0), rounded to bfloat16, two to a 32-bit column
            uint64_t la[4] = {0ull, 0ull, 0ull, 0ull};         // pairs of partial sums
            const uint64_t sc2 = pack2(sc, sc), mref2 = pack2(-mref, -mref);
            uint32_t pw[kKeys / 2];
#pragma unroll
            for (int x = 0; x < kKeys; x += 2) {
                float ea, eb;
                unpack2(fma2(pack2(__uint_as_float(v[x]), __uint_as_float(v[x + 1])), sc2, mref2), ea, eb);
                const float pa = fast_exp2(ea), pb = fast_exp2(eb);
                la[(x >> 1) & 3] = add2(la[(x >> 1) & 3], pack2(pa, pb));
                __nv_bfloat162 hb = __floats2bfloat162_rn(pa, pb);
                pw[x >> 1] = *reinterpret_cast<uint32_t*>(&hb);
            }
            {
                float s0, s1;
                unpack2(add2(add2(la[0], la[1]), add2(la[2], la[3])), s0, s1);
                l += s0 + s1;
            }
            // P goes where this tile's S was: every row of it that this warp owns is in registers
            tmem_st_32x32(ts + (uint32_t)((t & 1) * kKeys), pw);
            loaded = __shfl_sync(0xffffffffu, s_next, 0) != 0;
            if (loaded) {
                tc_fence_after();
#pragma unroll
                for (int c0 = 0; c0 < kKeys; c0 += 32)
                    tmem_ld_32x32(ts + (uint32_t)(((t + 1) & 1) * kKeys + c0), *reinterpret_cast<uint32_t(*)[32]>(&v[c0]));
            }
            tmem_st_wait();
            warp_arrive(&pf[t & 1], lane);
        }
        if (loaded) tmem_ld_wait();                            // (only after a wait that ran out)
        // all tiles issued: the last P V closes this map's accumulator
        if (ok) ok = warp_wait(&of[(n_tiles - 1) & 1], (uint32_t)((n_tiles - 1) >> 1) & 1, &abort_flag, lane);
        sL[m_ * kRows + il] = l > 0.f ? 1.f / l : 0.f;
        // both maps' warps meet (also after a wait that ran out): both accumulators are closed behind this
        tc_fence_before();
        asm volatile("bar.sync 1, 256;" ::: "memory");
        tc_fence_after();
        const bool whole = *reinterpret_cast<const volatile int*>(&abort_flag) == 0;
        // this map's warps take half of the value columns of both accumulators
        constexpr int HALF = V / 2;
        const float i0n = sL[il], i1n = sL[kRows + il] * prm.lambda[0];
        const uint32_t o0 = tmem + lane_sel + 2 * kKeys + (uint32_t)(m_ * HALF), o1 = o0 + kMapCols;
        float y[HALF], ss = 0.f;
#pragma unroll
        for (int c0 = 0; c0 < HALF; c0 += 32) {
            uint32_t a[32], b[32];
            tmem_ld_32x32(o0 + c0, a);
            tmem_ld_32x32(o1 + c0, b);
            tmem_ld_wait();
#pragma unroll
            for (int x = 0; x < 32; ++x) {
                y[c0 + x] = __uint_as_float(a[x]) * i0n - __uint_as_float(b[x]) * i1n;
                ss += y[c0 + x] * y[c0 + x];
            }
        }
        sSS[m_ * kRows + il] = ss;
        asm volatile("bar.sync 1, 256;" ::: "memory");
        const float mul = prm.post / sqrtf((sSS[il] + sSS[kRows + il]) / (float)prm.dv + prm.eps);
        if (live && whole) {
            bf16* dst = prm.out + ((size_t)(qs + i0 + il) * prm.nh + h) * prm.dv + m_ * HALF;
#pragma unroll
            for (int d = 0; d < HALF; d += 8) {
                if (m_ * HALF + d < prm.dv) {
                    uint32_t w[4];
#pragma unroll
                    for (int x = 0; x < 4; ++x) {
                        __nv_bfloat162 hb = __floats2bfloat162_rn(y[d + 2 * x] * mul, y[d + 2 * x + 1] * mul);
                        w[x] = *reinterpret_cast<uint32_t*>(&hb);
                    }
                    *reinterpret_cast<uint4*>(dst + d) = make_uint4(w[0], w[1], w[2], w[3]);
                }
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        tmem_dealloc(tmem, kTmemCols);
    }
}

// ------------------------------------------------------------------ host side
// Does this kernel take the case?  bf16 is implied by the caller.
LSB_API int lsb_prefill_attention_diff_tc5_supported(const void* q, const void* k_pages, const void* v_pages, const void* out,
                                                     int nh, int nkv, int dk, int dv, int page_size, float scale) {
    const bool pow2 = page_size > 0 && (page_size & (page_size - 1)) == 0;
    return dk > 0 && dk <= 128 && dk % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0 && nkv > 0 && nh % nkv == 0 && pow2 &&
           page_size >= 8 && page_size <= kKeys && scale > 0.f && ((uintptr_t)q % 16) == 0 && ((uintptr_t)k_pages % 16) == 0 &&
           ((uintptr_t)v_pages % 16) == 0 && ((uintptr_t)out % 16) == 0;
}

template <int D, int V>
static int launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const DiffTcParams& prm, dim3 grid,
                  cudaStream_t stream) {
    static int configured = -1;
    constexpr size_t smem = DiffSmem<D, V>::kTotal;
    static_assert(smem <= 227 * 1024, "a block's shared memory");
    if (configured < 0)
        configured = (int)cudaFuncSetAttribute(prefill_attention_diff_tc5_kernel<D, V>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (configured) return configured;
    return lsb_launch(prefill_attention_diff_tc5_kernel<D, V>, grid, dim3(kThreads), smem, stream, 1, mq, mk, mv, prm);
}

// q [tokens, nh * 2 * dk]; every request of the span is processed, single tokens as tiles of one row.
LSB_API int lsb_prefill_attention_diff_tc5(const void* q, int n_tokens, const void* k_pages, const void* v_pages,
                                           const int* q_start, const int* kv_len, const int* table_rows, const int* block_table,
                                           int table_stride, void* out, int n_requests, int max_q_len, int nh, int nkv, int dk,
                                           int dv, int page_size, int num_pages, float scale, int window, const float* lambda,
                                           float eps, float post, cudaStream_t stream) {
    if (n_requests <= 0 || max_q_len <= 0) return 0;
    if (!lsb_prefill_attention_diff_tc5_supported(q, k_pages, v_pages, out, nh, nkv, dk, dv, page_size, scale) || !lambda ||
        n_requests > 65535 || (max_q_len + kRows - 1) / kRows > 65535)
        return (int)cudaErrorInvalidValue;
    CUtensorMap mq, mk, mv;
    int rc;
    {
        cuuint64_t dims[3] = {(cuuint64_t)dk, (cuuint64_t)2 * nh, (cuuint64_t)n_tokens};
        cuuint64_t strides[2] = {(cuuint64_t)dk * 2, (cuuint64_t)nh * 2 * dk * 2};
        cuuint32_t box[3] = {64, 1, (cuuint32_t)kRows};
        if ((rc = encode(&mq, q, 3, dims, strides, box))) return rc;
    }
    {
        cuuint64_t dims[5] = {(cuuint64_t)dk, 2, (cuuint64_t)page_size, (cuuint64_t)nkv, (cuuint64_t)num_pages};
        cuuint64_t strides[4] = {(cuuint64_t)dk * 2, (cuuint64_t)2 * dk * 2, (cuuint64_t)page_size * 2 * dk * 2,
                                 (cuuint64_t)nkv * page_size * 2 * dk * 2};
        cuuint32_t box[5] = {64, 1, (cuuint32_t)page_size, 1, 1};
        if ((rc = encode(&mk, k_pages, 5, dims, strides, box))) return rc;
    }
    {
        cuuint64_t dims[4] = {(cuuint64_t)dv, (cuuint64_t)page_size, (cuuint64_t)nkv, (cuuint64_t)num_pages};
        cuuint64_t strides[3] = {(cuuint64_t)dv * 2, (cuuint64_t)page_size * dv * 2, (cuuint64_t)nkv * page_size * dv * 2};
        cuuint32_t box[4] = {64, (cuuint32_t)page_size, 1, 1};
        if ((rc = encode(&mv, v_pages, 4, dims, strides, box))) return rc;
    }
    DiffTcParams prm;
    prm.q_start = q_start; prm.kv_len = kv_len; prm.table_rows = table_rows; prm.block_table = block_table;
    prm.table_stride = table_stride; prm.out = (bf16*)out; prm.nh = nh; prm.nkv = nkv; prm.dv = dv;
    prm.page_size = page_size; prm.num_pages = num_pages; prm.scale = scale; prm.window = window;
    prm.lambda = lambda; prm.eps = eps; prm.post = post;
    int sh = 0;
    while ((1 << sh) < page_size) ++sh;
    prm.page_shift = sh;
    dim3 grid(nh, (max_q_len + kRows - 1) / kRows, n_requests);
    if (dk <= 64)
        return dv <= 64 ? launch<64, 64>(mq, mk, mv, prm, grid, stream) : launch<64, 128>(mq, mk, mv, prm, grid, stream);
    return dv <= 64 ? launch<128, 64>(mq, mk, mv, prm, grid, stream) : launch<128, 128>(mq, mk, mv, prm, grid, stream);
}
