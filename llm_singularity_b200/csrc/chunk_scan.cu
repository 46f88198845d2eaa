// Prompt portions of a matrix memory that fades by one number per head and token, on the tensor cores:
//
//     S_t = a_t S_(t-1) + w_t k_t v_t^T        o_t = S_t^T q_t        a_t, w_t numbers of the head
//
// The same recurrence as csrc/linear_scan.cu walks token by token, cut into chunks of 128 tokens.  With c_t
// the sum of log a over the chunk's tokens up to t:
//
//   chunk_gain     per chunk: E = sum_s exp(c_end - c_s) w_s k_s v_s^T, what the chunk adds to the state
//   chunk_chain    start(0) = the slot's state, start(j + 1) = exp(c_end of j) start(j) + E_j; the slot gets the
//                  state after the last chunk
//   chunk_output   o_t = exp(c_t) start^T q_t + sum_(s <= t) exp(c_t - c_s) w_s (q_t . k_s) v_s
//
// All three products of a token and the sums over a chunk run on mma.sync (bfloat16 operands, 32-bit sums).
// What is not a bfloat16 number already goes in as the sum of two (the rounded value and the rounded
// rest, 16 digits of mantissa): the states, the weighted keys, the weighted scores and, where they were
// rotated in 32-bit (SPLIT), queries and keys; so nothing of the recurrence is rounded to bfloat16's 8 digits.
// Sums of logarithms are formed in 64-bit and kept as pairs of floats: the difference of two of them is good
// to 32-bit however far the memory has faded.  Different chunks and heads are different blocks; the sums
// form in another order than in the walk: equal beyond rounding.
//
// rows: bfloat16 [tokens, ld]; a head's q, k and v at q_off, k_off (head h / share) and v_off (head h) with the rests
// of q and k (SPLIT) at q_lo and k_lo.  The state is [slot, head, V, N] 32-bit, N (channels of q and k)
// contiguous; N and V multiples of 8 up to 128.  Scratch: a row per chunk, chunk j of request r at
// q_start[r] / 128 + r + j.
#include "common.cuh"

LSB_DEFINE_STATUS()

typedef __nv_bfloat16 bf16;

constexpr int kL = 128;                  // tokens of a chunk
constexpr int kThreads = 256;

struct ChunkArgs {
    const bf16* rows; long long ld;
    int q_off, k_off, v_off, q_lo, k_lo;
    int heads, share, N, V;
    const float *log_keep, *write;       // [tokens, heads] (null: log_fixed, and 1)
    const float* log_fixed;              // [heads]
    float q_scale;
    float* state; int n_slots;
    const int *q_start, *table_rows;
    float* gain;                         // [chunk, heads, V, N]
    float* fade;                         // [chunk, heads]: the chunk's whole decay
    bf16* starts;                        // [chunk, heads, 2, V, N]: rounded start state, rounded rest
    float* out;                          // [tokens, heads * V]
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4_t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void copy16(void* dst, const void* src, bool real) {
    const int n = real ? 16 : 0;         // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ uint32_t pack2(float lo, float hi) {
    __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}
// two floats as pairs of bfloat16: the rounded values, and the rounded rests
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack2(a, b);
    lo = pack2(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}

// c of every token of the chunk (base-2 logarithm, a pair of floats) and its write factor into shared memory;
// tokens past the chunk's end keep the last sum and write nothing.  Warp 0; the caller synchronises.
__device__ __forceinline__ void chunk_sums(const ChunkArgs& a, int t0, int n, int h, float2* cum, float* wr) {
    const int lane = threadIdx.x;
    double v[4];
    double run = 0.0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int s = lane * 4 + i;
        float la = 0.f, w = 0.f;
        if (s < n) {
            la = a.log_keep ? a.log_keep[(size_t)(t0 + s) * a.heads + h] : a.log_fixed[h];
            w = a.write ? a.write[(size_t)(t0 + s) * a.heads + h] : 1.f;
        }
        wr[s] = w;
        run += (double)fmaxf(la, -1000.f) * 1.4426950408889634;      // (2^-1443 is zero already)
        v[i] = run;
    }
    double sum = run;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double below = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += below;
    }
    const double before = sum - run;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const double c = before + v[i];
        const float hi = (float)c;
        cum[lane * 4 + i] = make_float2(hi, (float)(c - (double)hi));
    }
}
// exp of the difference of two such sums
__device__ __forceinline__ float faded(const float2& later, const float2& earlier) {
    return exp2f((later.x - earlier.x) + (later.y - earlier.y));
}

struct Where { int r, sg, t0, n; size_t row; bool live; };
__device__ __forceinline__ Where chunk_of(const ChunkArgs& a) {
    Where w;
    w.r = blockIdx.z;
    w.sg = blockIdx.x;
    const int q0 = a.q_start[w.r], q1 = a.q_start[w.r + 1];
    w.t0 = q0 + w.sg * kL;
    w.n = min(kL, q1 - w.t0);
    w.row = (size_t)(q0 / kL + w.r + w.sg);
    w.live = w.n > 0;
    return w;
}

template <int NP, int VP, bool SPLIT>
__global__ void __launch_bounds__(kThreads) chunk_gain_kernel(ChunkArgs a) {
    constexpr int KS = NP + 8, VS = VP + 8;                     // row strides: four words past a multiple of 32
    extern __shared__ __align__(16) unsigned char sm[];
    bf16* k_hi = reinterpret_cast<bf16*>(sm);                   // [kL][KS], weighted keys
    bf16* k_lo = k_hi + kL * KS;
    bf16* vs = k_lo + kL * KS;                                  // [kL][VS]
    __shared__ float2 cum[kL];
    __shared__ float wr[kL];
    lsb_pdl_launch_dependents();
    const Where at = chunk_of(a);                               // (metadata of the step)
    if (!at.live) return;
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    lsb_pdl_wait();
    constexpr int VG = VP / 8, NG = NP / 8;
    for (int w = threadIdx.x; w < kL * VG; w += kThreads) {
        const int s = w / VG, c = (w - s * VG) * 8;
        const bool real = s < at.n && c < a.V;
        copy16(vs + s * VS + c, a.rows + (real ? (size_t)(at.t0 + s) * a.ld + a.v_off + h * a.V + c : 0), real);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (warp == 0) chunk_sums(a, at.t0, at.n, h, cum, wr);
    __syncthreads();
    const float2 end = cum[kL - 1];
    const int hk = h / a.share;
    for (int w = threadIdx.x; w < kL * NG; w += kThreads) {
        const int s = w / NG, c = (w - s * NG) * 8;
        uint4 hi = make_uint4(0u, 0u, 0u, 0u), lo = hi;
        if (s < at.n && c < a.N) {
            const bf16* src = a.rows + (size_t)(at.t0 + s) * a.ld + hk * a.N + c;
            const float f = faded(end, cum[s]) * wr[s];
            const uint4 raw = *reinterpret_cast<const uint4*>(src + a.k_off);
            uint4 rest = make_uint4(0u, 0u, 0u, 0u);
            if (SPLIT) rest = *reinterpret_cast<const uint4*>(src + a.k_lo);
            const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
            const __nv_bfloat162* q = reinterpret_cast<const __nv_bfloat162*>(&rest);
            uint32_t* ph = reinterpret_cast<uint32_t*>(&hi);
            uint32_t* pl = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                float2 x = __bfloat1622float2(p[j]);
                if (SPLIT) {
                    const float2 y = __bfloat1622float2(q[j]);
                    x.x += y.x;
                    x.y += y.y;
                }
                split2(x.x * f, x.y * f, ph[j], pl[j]);
            }
        }
        *reinterpret_cast<uint4*>(k_hi + s * KS + c) = hi;
        *reinterpret_cast<uint4*>(k_lo + s * KS + c) = lo;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // E [V, N]: a warp has 16 rows of V and all of N, or half of N where V is 64
    constexpr int WN = VP == 128 ? NP : NP / 2;
    const int v0 = (VP == 128 ? warp : warp & 3) * 16, n0 = VP == 128 ? 0 : (warp >> 2) * WN;
    float e[WN / 8][4];
#pragma unroll
    for (int j = 0; j < WN / 8; ++j) e[j][0] = e[j][1] = e[j][2] = e[j][3] = 0.f;
    if (v0 < a.V && n0 < a.N) {
        const int i8 = lane >> 3, l8 = lane & 7;
        const uint32_t va = smem_u32(vs + ((i8 >> 1) * 8 + l8) * VS + v0 + (i8 & 1) * 8);
        const uint32_t ka = smem_u32(k_hi + ((i8 & 1) * 8 + l8) * KS + n0 + (i8 >> 1) * 8);
        const int steps = (at.n + 15) >> 4;
        for (int ks = 0; ks < steps; ++ks) {
            uint32_t fa[4];
            ldsm4_t(fa, va + ks * 16 * VS * 2);
#pragma unroll
            for (int j = 0; j < WN / 16; ++j) {
                uint32_t b[4], c[4];
                const uint32_t addr = ka + ks * 16 * KS * 2 + j * 32;
                ldsm4_t(b, addr);
                ldsm4_t(c, addr + kL * KS * 2);
                mma16816(e[2 * j], fa, b[0], b[1]);
                mma16816(e[2 * j + 1], fa, b[2], b[3]);
                mma16816(e[2 * j], fa, c[0], c[1]);
                mma16816(e[2 * j + 1], fa, c[2], c[3]);
            }
        }
        float* dst = a.gain + (at.row * a.heads + h) * (size_t)a.V * a.N;
        const int gid = lane >> 2, tid4 = lane & 3;
#pragma unroll
        for (int j = 0; j < WN / 8; ++j) {
            const int n = n0 + j * 8 + 2 * tid4;
            if (n < a.N) {
                if (v0 + gid < a.V) *reinterpret_cast<float2*>(dst + (size_t)(v0 + gid) * a.N + n) = make_float2(e[j][0], e[j][1]);
                if (v0 + gid + 8 < a.V) *reinterpret_cast<float2*>(dst + (size_t)(v0 + gid + 8) * a.N + n) = make_float2(e[j][2], e[j][3]);
            }
        }
    }
    if (threadIdx.x == 0) a.fade[at.row * a.heads + h] = exp2f(end.x + end.y);
}

constexpr int kChainThreads = 128;

__global__ void __launch_bounds__(kChainThreads) chunk_chain_kernel(ChunkArgs a) {
    lsb_pdl_launch_dependents();
    const int r = blockIdx.z, h = blockIdx.y;
    const int q0 = a.q_start[r], len = a.q_start[r + 1] - q0;
    const int slot = a.table_rows[r];
    if (len <= 0) return;
    if (slot < 0 || slot >= a.n_slots) {
        if (threadIdx.x == 0) lsb_set_status(LSB_BAD_ROW);
        return;
    }
    const int chunks = (len + kL - 1) / kL;
    const size_t row0 = (size_t)(q0 / kL + r), per = (size_t)a.V * a.N;
    const size_t i = ((size_t)blockIdx.x * kChainThreads + threadIdx.x) * 4;
    if (i >= per) return;
    lsb_pdl_wait();
    float* st = a.state + ((size_t)slot * a.heads + h) * per + i;
    float4 cur = *reinterpret_cast<const float4*>(st);
    constexpr int kAhead = 8;
    for (int s0 = 0; s0 < chunks; s0 += kAhead) {              // eight chunks' loads in flight at once
        float4 e[kAhead];
        float f[kAhead];
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            const size_t hr = (row0 + min(s0 + k, chunks - 1)) * a.heads + h;
            e[k] = *reinterpret_cast<const float4*>(a.gain + hr * per + i);
            f[k] = a.fade[hr];
        }
#pragma unroll
        for (int k = 0; k < kAhead; ++k) {
            if (s0 + k < chunks) {
                bf16* dst = a.starts + ((row0 + s0 + k) * a.heads + h) * 2 * per + i;
                uint2 hi, lo;
                split2(cur.x, cur.y, hi.x, lo.x);
                split2(cur.z, cur.w, hi.y, lo.y);
                *reinterpret_cast<uint2*>(dst) = hi;
                *reinterpret_cast<uint2*>(dst + per) = lo;
                cur.x = f[k] * cur.x + e[k].x;
                cur.y = f[k] * cur.y + e[k].y;
                cur.z = f[k] * cur.z + e[k].z;
                cur.w = f[k] * cur.w + e[k].w;
            }
        }
    }
    *reinterpret_cast<float4*>(st) = cur;
}

template <int NP, int VP, bool SPLIT>
__global__ void __launch_bounds__(kThreads) chunk_output_kernel(ChunkArgs a) {
    constexpr int KS = NP + 8, VS = VP + 8;
    extern __shared__ __align__(16) unsigned char sm[];
    bf16* s_hi = reinterpret_cast<bf16*>(sm);                   // [VP][KS] start state
    bf16* s_lo = s_hi + VP * KS;
    bf16* k_hi = s_lo + VP * KS;                                // [kL][KS]
    bf16* k_lo = k_hi + (SPLIT ? kL * KS : 0);
    bf16* vs = k_lo + kL * KS;                                  // [kL][VS]
    __shared__ float2 cum[kL];
    __shared__ float wr[kL];
    lsb_pdl_launch_dependents();
    const Where at = chunk_of(a);
    if (!at.live) return;
    const int h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tid4 = lane & 3;
    lsb_pdl_wait();
    constexpr int VG = VP / 8, NG = NP / 8;
    const int hk = h / a.share;
    const size_t per = (size_t)a.V * a.N;
    const bf16* start = a.starts + (at.row * a.heads + h) * 2 * per;
    for (int w = threadIdx.x; w < VP * NG; w += kThreads) {
        const int v = w / NG, c = (w - v * NG) * 8;
        const bool real = v < a.V && c < a.N;
        copy16(s_hi + v * KS + c, start + (real ? (size_t)v * a.N + c : 0), real);
        copy16(s_lo + v * KS + c, start + (real ? per + (size_t)v * a.N + c : 0), real);
    }
    for (int w = threadIdx.x; w < kL * NG; w += kThreads) {
        const int s = w / NG, c = (w - s * NG) * 8;
        const bool real = s < at.n && c < a.N;
        const bf16* src = a.rows + (real ? (size_t)(at.t0 + s) * a.ld + hk * a.N + c : 0);
        copy16(k_hi + s * KS + c, src + (real ? a.k_off : 0), real);
        if (SPLIT) copy16(k_lo + s * KS + c, src + (real ? a.k_lo : 0), real);
    }
    for (int w = threadIdx.x; w < kL * VG; w += kThreads) {
        const int s = w / VG, c = (w - s * VG) * 8;
        const bool real = s < at.n && c < a.V;
        copy16(vs + s * VS + c, a.rows + (real ? (size_t)(at.t0 + s) * a.ld + a.v_off + h * a.V + c : 0), real);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (warp == 0) chunk_sums(a, at.t0, at.n, h, cum, wr);
    const int row_a = warp * 16 + gid, row_b = row_a + 8;      // this thread's two tokens of the chunk
    const bool ok_a = row_a < at.n, ok_b = row_b < at.n;
    uint32_t q[NP / 16][4], ql[SPLIT ? NP / 16 : 1][4];
    {
        const bf16* qa = a.rows + (size_t)(at.t0 + (ok_a ? row_a : 0)) * a.ld + hk * a.N;
        const bf16* qb = a.rows + (size_t)(at.t0 + (ok_b ? row_b : 0)) * a.ld + hk * a.N;
#pragma unroll
        for (int ks = 0; ks < NP / 16; ++ks) {
            const int c = ks * 16 + 2 * tid4;
            const bool in0 = c < a.N, in1 = c + 8 < a.N;
            q[ks][0] = ok_a && in0 ? *reinterpret_cast<const uint32_t*>(qa + a.q_off + c) : 0u;
            q[ks][1] = ok_b && in0 ? *reinterpret_cast<const uint32_t*>(qb + a.q_off + c) : 0u;
            q[ks][2] = ok_a && in1 ? *reinterpret_cast<const uint32_t*>(qa + a.q_off + c + 8) : 0u;
            q[ks][3] = ok_b && in1 ? *reinterpret_cast<const uint32_t*>(qb + a.q_off + c + 8) : 0u;
            if (SPLIT) {
                ql[SPLIT ? ks : 0][0] = ok_a && in0 ? *reinterpret_cast<const uint32_t*>(qa + a.q_lo + c) : 0u;
                ql[SPLIT ? ks : 0][1] = ok_b && in0 ? *reinterpret_cast<const uint32_t*>(qb + a.q_lo + c) : 0u;
                ql[SPLIT ? ks : 0][2] = ok_a && in1 ? *reinterpret_cast<const uint32_t*>(qa + a.q_lo + c + 8) : 0u;
                ql[SPLIT ? ks : 0][3] = ok_b && in1 ? *reinterpret_cast<const uint32_t*>(qb + a.q_lo + c + 8) : 0u;
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (warp * 16 >= at.n) return;
    const float2 ca = cum[row_a], cb = cum[row_b];
    float o[VP / 8][4];
#pragma unroll
    for (int j = 0; j < VP / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    const int i8 = lane >> 3, l8 = lane & 7;
    {
        // what the chunk found: start^T q
        const uint32_t sa = smem_u32(s_hi + ((i8 >> 1) * 8 + l8) * KS + (i8 & 1) * 8);
#pragma unroll
        for (int ks = 0; ks < NP / 16; ++ks) {
#pragma unroll
            for (int j = 0; j < VP / 16; ++j) {
                uint32_t b[4], c[4];
                const uint32_t addr = sa + (j * 16 * KS + ks * 16) * 2;
                ldsm4(b, addr);
                ldsm4(c, addr + VP * KS * 2);
                mma16816(o[2 * j], q[ks], b[0], b[1]);
                mma16816(o[2 * j + 1], q[ks], b[2], b[3]);
                mma16816(o[2 * j], q[ks], c[0], c[1]);
                mma16816(o[2 * j + 1], q[ks], c[2], c[3]);
                if (SPLIT) {
                    mma16816(o[2 * j], ql[SPLIT ? ks : 0], b[0], b[1]);
                    mma16816(o[2 * j + 1], ql[SPLIT ? ks : 0], b[2], b[3]);
                }
            }
        }
    }
    // What the chunk's own tokens wrote, sixteen of them at a time up to this warp's.  What came before the warp's
    // first token fades to it first (one factor per earlier token, and one for the start state) and from there
    // with the row (one factor at the end): both are at most 1, so nothing overflows on the way.
    const float2 ref = cum[warp * 16];
    {
        const float f = exp2f(ref.x + ref.y);
#pragma unroll
        for (int j = 0; j < VP / 8; ++j) {
            o[j][0] *= f;
            o[j][1] *= f;
            o[j][2] *= f;
            o[j][3] *= f;
        }
    }
    const uint32_t ka = smem_u32(k_hi + ((i8 >> 1) * 8 + l8) * KS + (i8 & 1) * 8);
    const uint32_t va = smem_u32(vs + ((i8 & 1) * 8 + l8) * VS + (i8 >> 1) * 8);
    for (int g = 0; g <= warp; ++g) {
        if (g == warp) {
            const float fa = faded(ca, ref) * a.q_scale, fb = faded(cb, ref) * a.q_scale;
#pragma unroll
            for (int j = 0; j < VP / 8; ++j) {
                o[j][0] *= fa;
                o[j][1] *= fa;
                o[j][2] *= fb;
                o[j][3] *= fb;
            }
        }
        float s[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < NP / 16; ++ks) {
            uint32_t b[4];
            const uint32_t addr = ka + (g * 16 * KS + ks * 16) * 2;
            ldsm4(b, addr);
            mma16816(s[0], q[ks], b[0], b[1]);
            mma16816(s[1], q[ks], b[2], b[3]);
            if (SPLIT) {
                uint32_t c[4];
                ldsm4(c, addr + kL * KS * 2);
                mma16816(s[0], ql[SPLIT ? ks : 0], b[0], b[1]);
                mma16816(s[1], ql[SPLIT ? ks : 0], b[2], b[3]);
                mma16816(s[0], q[ks], c[0], c[1]);
                mma16816(s[1], q[ks], c[2], c[3]);
            }
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int t = g * 16 + j * 8 + 2 * tid4;
            const float2 c0 = cum[t], c1 = cum[t + 1];
            float p0, p1, p2, p3;
            if (g < warp) {
                const float f0 = faded(ref, c0) * wr[t], f1 = faded(ref, c1) * wr[t + 1];
                p0 = s[j][0] * f0;
                p1 = s[j][1] * f1;
                p2 = s[j][2] * f0;
                p3 = s[j][3] * f1;
            } else {
                const float w0 = wr[t] * a.q_scale, w1 = wr[t + 1] * a.q_scale;
                p0 = t <= row_a ? s[j][0] * (faded(ca, c0) * w0) : 0.f;
                p1 = t + 1 <= row_a ? s[j][1] * (faded(ca, c1) * w1) : 0.f;
                p2 = t <= row_b ? s[j][2] * (faded(cb, c0) * w0) : 0.f;
                p3 = t + 1 <= row_b ? s[j][3] * (faded(cb, c1) * w1) : 0.f;
            }
            split2(p0, p1, ph[2 * j], pl[2 * j]);
            split2(p2, p3, ph[2 * j + 1], pl[2 * j + 1]);
        }
#pragma unroll
        for (int j = 0; j < VP / 16; ++j) {
            uint32_t b[4];
            ldsm4_t(b, va + (g * 16 * VS + j * 16) * 2);
            mma16816(o[2 * j], ph, b[0], b[1]);
            mma16816(o[2 * j + 1], ph, b[2], b[3]);
            mma16816(o[2 * j], pl, b[0], b[1]);
            mma16816(o[2 * j + 1], pl, b[2], b[3]);
        }
    }
    const size_t ldo = (size_t)a.heads * a.V;
    float* oa = a.out + (size_t)(at.t0 + row_a) * ldo + (size_t)h * a.V;
    float* ob = a.out + (size_t)(at.t0 + row_b) * ldo + (size_t)h * a.V;
#pragma unroll
    for (int j = 0; j < VP / 8; ++j) {
        const int c = j * 8 + 2 * tid4;
        if (c < a.V) {
            if (ok_a) *reinterpret_cast<float2*>(oa + c) = make_float2(o[j][0], o[j][1]);
            if (ok_b) *reinterpret_cast<float2*>(ob + c) = make_float2(o[j][2], o[j][3]);
        }
    }
}

// ------------------------------------------------------------------ operands of a rotated memory
// From the 32-bit rows of a projection to the rows of the kernels above: q and k turned by the token's
// position (pairs (i, i + dims / 2) of the first `dims` channels of every head, angle and rotation in 32-bit), each
// as a rounded value and a rounded rest, and v rounded: [q | rest of q | k | rest of k | v].
constexpr int kTurnMaxHalf = 512;

__global__ void __launch_bounds__(256) turn_split_kernel(const float* __restrict__ proj, long long ld, int q_off, int k_off, int v_off,
                                                         int heads, int D, int vv, int dims, const float* __restrict__ inv_freq,
                                                         const int* __restrict__ positions, int first, bf16* __restrict__ rows) {
    __shared__ float cs[kTurnMaxHalf], sn[kTurnMaxHalf];
    lsb_pdl_launch_dependents();
    const int t = blockIdx.x + first, half = dims >> 1, qk = heads * D;
    const float pos = (float)positions[t];
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * inv_freq[i], &sn[i], &cs[i]);
    __syncthreads();
    lsb_pdl_wait();
    const float* src = proj + (size_t)t * ld;
    bf16* dst = rows + (size_t)t * (4 * qk + vv);
    const int pairs = D >> 1, per = 2 * heads * pairs;
    for (int w = threadIdx.x; w < per; w += blockDim.x) {
        const int hh = w / pairs, i = w - hh * pairs;
        const bool is_q = hh < heads;
        const int hd = (is_q ? hh : hh - heads) * D;
        // the turning pairs first, then the rest two by two
        const int ia = i < half ? i : dims + 2 * (i - half), ib = i < half ? i + half : ia + 1;
        const float* x = src + (is_q ? q_off : k_off) + hd;
        float a = x[ia], b = x[ib];
        if (i < half) {
            const float u = a * cs[i] - b * sn[i];
            b = b * cs[i] + a * sn[i];
            a = u;
        }
        bf16* o = dst + (is_q ? 0 : 2 * qk) + hd;
        const bf16 ha = __float2bfloat16_rn(a), hb = __float2bfloat16_rn(b);
        o[ia] = ha;
        o[ib] = hb;
        o[qk + ia] = __float2bfloat16_rn(a - __bfloat162float(ha));
        o[qk + ib] = __float2bfloat16_rn(b - __bfloat162float(hb));
    }
    for (int w = threadIdx.x * 2; w < vv; w += blockDim.x * 2)
        *reinterpret_cast<__nv_bfloat162*>(dst + 4 * qk + w) = __floats2bfloat162_rn(src[v_off + w], src[v_off + w + 1]);
}

// tokens first .. first + tokens - 1 of the step
LSB_API int lsb_turn_split(const float* proj, long long ld, int q_off, int k_off, int v_off, int heads, int D, int vv, int dims,
                           const float* inv_freq, const int* positions, int first, int tokens, void* rows, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (heads <= 0 || D <= 0 || D % 2 || vv % 2 || dims < 0 || dims % 2 || dims > D || dims / 2 > kTurnMaxHalf || first < 0)
        return (int)cudaErrorInvalidValue;
    return lsb_launch(turn_split_kernel, dim3(tokens), dim3(256), 0, stream, 1, proj, ld, q_off, k_off, v_off, heads, D, vv, dims,
                      inv_freq, positions, first, (bf16*)rows);
}

// ------------------------------------------------------------------ host side
LSB_API int lsb_chunk_tokens() { return kL; }

LSB_API int lsb_chunk_scan_supported(int N, int V) { return N > 0 && V > 0 && N % 8 == 0 && V % 8 == 0 && N <= 128 && V <= 128; }

template <int NP, int VP, bool SPLIT>
static int run_chunks(const ChunkArgs& a, int n_requests, int chunks, cudaStream_t stream) {
    constexpr int KS = NP + 8, VS = VP + 8;
    constexpr size_t gain_sm = (size_t)(2 * kL * KS + kL * VS) * sizeof(bf16);
    constexpr size_t out_sm = (size_t)(2 * VP * KS + (SPLIT ? 2 : 1) * kL * KS + kL * VS) * sizeof(bf16);
    static int configured = -1;
    if (configured < 0) {
        configured = (int)cudaFuncSetAttribute(chunk_gain_kernel<NP, VP, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gain_sm);
        if (!configured)
            configured = (int)cudaFuncSetAttribute(chunk_output_kernel<NP, VP, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_sm);
    }
    if (configured) return configured;
    dim3 grid(chunks, a.heads, n_requests);
    int rc = lsb_launch(chunk_gain_kernel<NP, VP, SPLIT>, grid, dim3(kThreads), gain_sm, stream, 1, a);
    if (rc) return rc;
    const int per = a.V * a.N / 4;
    rc = lsb_launch(chunk_chain_kernel, dim3((per + kChainThreads - 1) / kChainThreads, a.heads, n_requests), dim3(kChainThreads), 0,
                    stream, 1, a);
    if (rc) return rc;
    return lsb_launch(chunk_output_kernel<NP, VP, SPLIT>, grid, dim3(kThreads), out_sm, stream, 1, a);
}

// log_keep and write [tokens, heads] (both or neither), else log_fixed [heads]; q_lo, k_lo >= 0: queries and keys are split.
// gain, starts, fade: scratch of tokens / 128 + requests rows (see above).  q_start and table_rows begin at the
// first request to be run.
LSB_API int lsb_chunk_scan(const void* rows, long long ld, int q_off, int k_off, int v_off, int q_lo, int k_lo, int heads,
                           int key_heads, int N, int V, const float* log_keep, const float* write, const float* log_fixed,
                           float q_scale, float* state, int n_slots, const int* q_start, const int* table_rows, int n_requests,
                           int max_q_len, float* out, float* gain, void* starts, float* fade, cudaStream_t stream) {
    if (n_requests <= 0 || max_q_len <= 0) return 0;
    const bool split = q_lo >= 0;
    if (!lsb_chunk_scan_supported(N, V) || heads <= 0 || key_heads <= 0 || heads % key_heads || heads > 65535 || n_requests > 65535 ||
        (split != (k_lo >= 0)) || (!log_keep && !log_fixed) || (log_keep && !write) || !gain || !starts || !fade)
        return (int)cudaErrorInvalidValue;
    if ((uintptr_t)rows % 16 || ld % 8 || q_off % 8 || k_off % 8 || v_off % 8 || (split && (q_lo % 8 || k_lo % 8)) ||
        (uintptr_t)state % 16 || (uintptr_t)gain % 16 || (uintptr_t)starts % 16 || (uintptr_t)out % 8)
        return (int)cudaErrorInvalidValue;
    ChunkArgs a;
    a.rows = (const bf16*)rows; a.ld = ld;
    a.q_off = q_off; a.k_off = k_off; a.v_off = v_off; a.q_lo = q_lo; a.k_lo = k_lo;
    a.heads = heads; a.share = heads / key_heads; a.N = N; a.V = V;
    a.log_keep = log_keep; a.write = write; a.log_fixed = log_fixed; a.q_scale = q_scale;
    a.state = state; a.n_slots = n_slots; a.q_start = q_start; a.table_rows = table_rows;
    a.gain = gain; a.fade = fade; a.starts = (bf16*)starts; a.out = out;
    const int chunks = (max_q_len + kL - 1) / kL;
#define LSB_CHUNKS(NP, VP)                                                           \
    do {                                                                             \
        if (split) return run_chunks<NP, VP, true>(a, n_requests, chunks, stream);   \
        return run_chunks<NP, VP, false>(a, n_requests, chunks, stream);             \
    } while (0)
    if (N <= 64) {
        if (V <= 64) LSB_CHUNKS(64, 64);
        else LSB_CHUNKS(64, 128);
    } else {
        if (V <= 64) LSB_CHUNKS(128, 64);
        else LSB_CHUNKS(128, 128);
    }
#undef LSB_CHUNKS
    return 0;
}
