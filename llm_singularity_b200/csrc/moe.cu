// Routed experts: choosing, sorting rows by expert, the two grouped products and the sum.
//
//   moe_route    per token: scores from the 32-bit router logits (sigmoid, softmax over all experts,
//                or softmax over the chosen alone), the `top` largest (the lower index wins a tie),
//                optionally divided by their sum -> ids [T, top], weights [T, top].
//                (or no router: the experts of a token stand in a table's row of its id, all with one weight)
//   moe_align    the (token, choice) pairs sorted by expert into rows; each expert's rows start
//                on a multiple of the row tile, so a tile of rows belongs to one expert.  Writes
//                pos [T * top] (the row of each pair), row_token / row_scale [capacity] (-1 / 0 in
//                the padding) and tile_expert [capacity / tile] (-1 beyond the last used tile).
//   moe_up       rows gathered from x (times the row's weight if the weight goes on the input),
//                times the expert's gate/up matrix (rows alternate gate_i, up_i), act(g) * u; or
//                times its up matrix alone, act(u).
//   moe_down     times the expert's down matrix -> y [capacity, hidden] 32-bit.
//   moe_combine  out[t] = sum over the token's choices of y[pos] (times the weight if it goes on
//                the output), plus a shared expert's row (times a sigmoid), rounded to T once.
//
// Each output row depends only on its own input row and its expert's weights, and the sum runs
// over a token's choices in their order, so where a row landed does not change any result.
#include "common.cuh"

#include <float.h>

LSB_DEFINE_STATUS()

constexpr int kTile = 32;               // rows per tile; an expert's rows are padded to this

// act(g) * u of a gated expert; act 5 is the capped form with a limit L: min(g, L) sigmoid(1.702 min(g, L))
// (clamp(u, -L, L) + 1)
__device__ __forceinline__ float moe_gate_mul(float z, float up, int act, float limit) {
    if (act == 5) {
        const float g = fminf(z, limit);
        return g / (1.f + expf(-1.702f * g)) * (fminf(fmaxf(up, -limit), limit) + 1.f);
    }
    if (act == 1) return z / (1.f + expf(-z)) * up;
    if (act == 2) return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * up;
    return z * up;
}

// The activation of an ungated expert: 1 silu, 2 gelu in its tanh form, 6 the square of relu, else none.
__device__ __forceinline__ float moe_plain(float z, int act) {
    if (act == 6) {
        z = fmaxf(z, 0.f);
        return z * z;
    }
    return moe_gate_mul(z, 1.f, act, 0.f);
}

// How scores are made and weighted: `score` 0 sigmoid, 1 softmax over all experts, 2 softmax over the chosen
// logits alone; `bias` (one number an expert, may be null) is added to the scores for the choice only, or,
// with `joins`, to the logits themselves; the chosen scores are divided by their sum + eps if `renorm`,
// and multiplied by `scale`.  A token's logits are `ld` numbers apart.
struct RouteOpts {
    int score, renorm;
    const float* bias;
    float scale, eps;
    int joins, ld;
};

constexpr int kMaxTop = 32;

// Experts chosen by the token's id: tables [rows, top], every choice with the same weight.  Several layers'
// tables are worked through by a launch, a block each, since nothing but the tokens decides.
constexpr int kMaxTables = 32;

struct TokenRows {
    const int* tables[kMaxTables];
    const int* token_ids;
    int rows;
    float weight;
};

// One warp chooses for one token, up to 128 experts: the logits in registers, four a lane, a chosen one struck
// out; lane k keeps what the k-th choice was.
__device__ __forceinline__ void route_token_small(const float* __restrict__ z, int E, int top, const RouteOpts& ro,
                                                  int* __restrict__ ids, float* __restrict__ wts, int lane) {
    float zv[4], cv[4], zmax = -FLT_MAX, denom = 1.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int e = lane + 32 * i;
        zv[i] = -FLT_MAX;
        if (e < E) zv[i] = ro.joins && ro.bias ? z[e] + ro.bias[e] : z[e];
        zmax = fmaxf(zmax, zv[i]);
    }
    zmax = lsb_warp_max(zmax);
    if (ro.score == 1) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) s += lane + 32 * i < E ? expf(zv[i] - zmax) : 0.f;
        denom = lsb_warp_sum(s);
    }
    auto score_of = [&](float v) {          // (score 2: relative to the largest logit, which is always chosen)
        return ro.score == 0 ? 1.f / (1.f + expf(-v)) : expf(v - zmax) / denom;
    };
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int e = lane + 32 * i;
        cv[i] = e < E ? (ro.bias && !ro.joins ? score_of(zv[i]) + ro.bias[e] : zv[i]) : -FLT_MAX;
    }
    unsigned gone = 0;                      // bit i: this lane's i-th expert is chosen (or there is none)
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (lane + 32 * i >= E) gone |= 1u << i;
    float mine = 0.f, total = 0.f;
    int my_id = 0;
    for (int k = 0; k < top; ++k) {
        float best = -FLT_MAX, bz = 0.f;
        int bi = 0x7fffffff;
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (!(gone >> i & 1) && (bi == 0x7fffffff || cv[i] > best)) { best = cv[i]; bz = zv[i]; bi = lane + 32 * i; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o), oz = __shfl_xor_sync(0xffffffffu, bz, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (oi != 0x7fffffff && (bi == 0x7fffffff || ob > best || (ob == best && oi < bi))) { best = ob; bz = oz; bi = oi; }
        }
        if ((bi & 31) == lane) gone |= 1u << (bi >> 5);
        const float v = score_of(bz);
        if (lane == k) { mine = v; my_id = bi; }
        total += v;
    }
    if (lane < top) {
        ids[lane] = my_id;
        wts[lane] = (ro.score == 2 ? mine / total : ro.renorm ? mine / (total + ro.eps) : mine) * ro.scale;
    }
}

// One warp chooses for one token (all lanes call it together).
__device__ __forceinline__ void route_token(const float* __restrict__ z, int E, int top, const RouteOpts ro,
                                            int* __restrict__ ids, float* __restrict__ wts, int lane) {
    if (E <= 128) {
        route_token_small(z, E, top, ro, ids, wts, lane);
        return;
    }
    const int score = ro.score, renorm = ro.renorm;
    const float* add = ro.joins ? ro.bias : nullptr;         // part of the logits
    const float* correct = ro.joins ? nullptr : ro.bias;     // for the choice alone
    auto logit = [&](int e) { return add ? z[e] + add[e] : z[e]; };
    float zmax = -FLT_MAX, denom = 1.f;
    if (score == 1) {
        for (int e = lane; e < E; e += 32) zmax = fmaxf(zmax, logit(e));
        zmax = lsb_warp_max(zmax);
        float s = 0.f;
        for (int e = lane; e < E; e += 32) s += expf(logit(e) - zmax);
        denom = lsb_warp_sum(s);
    }
    int chosen[kMaxTop];
    float val[kMaxTop];
    float total = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -FLT_MAX;
        int bi = 0x7fffffff;
        for (int e = lane; e < E; e += 32) {
            bool taken = false;
            for (int j = 0; j < k; ++j) taken |= (chosen[j] == e);
            // (without a bias the logits order the experts as their scores do)
            const float c = correct ? (score == 1 ? expf(z[e] - zmax) / denom : 1.f / (1.f + expf(-z[e]))) + correct[e] : logit(e);
            if (!taken && (c > best || (c == best && e < bi))) { best = c; bi = e; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
        }
        chosen[k] = bi;
        if (correct) best = z[bi];
        if (score == 2) {                   // (the first chosen is the largest)
            if (k == 0) zmax = best;
            val[k] = expf(best - zmax);
        } else val[k] = score == 1 ? expf(best - zmax) / denom : 1.f / (1.f + expf(-best));
        total += val[k];
    }
    if (lane == 0) {
        for (int k = 0; k < top; ++k) {
            ids[k] = chosen[k];
            wts[k] = (score == 2 ? val[k] / total : renorm ? val[k] / (total + ro.eps) : val[k]) * ro.scale;
        }
    }
}

__global__ void moe_route_kernel(const float* __restrict__ logits, int n_tokens, int E, int top,
                                 RouteOpts ro, int* __restrict__ ids, float* __restrict__ wts) {
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int warp = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (warp >= n_tokens) return;
    route_token(logits + (size_t)warp * ro.ld, E, top, ro, ids + (size_t)warp * top, wts + (size_t)warp * top, lane);
}

__global__ void __launch_bounds__(1024, 1)
moe_align_kernel(int* __restrict__ ids, float* __restrict__ wts, int n, int top, int E,
                 int cap_tiles, int tile, int* __restrict__ pos, int* __restrict__ row_token,
                 float* __restrict__ row_scale, int* __restrict__ tile_expert,
                 const float* __restrict__ logits, RouteOpts ro, TokenRows by) {
    extern __shared__ int shi[];
    const int layer = blockIdx.x;
    ids += (size_t)layer * n;
    wts += (size_t)layer * n;
    pos += (size_t)layer * n;
    row_token += (size_t)layer * cap_tiles * tile;
    row_scale += (size_t)layer * cap_tiles * tile;
    tile_expert += (size_t)layer * cap_tiles;
    const int* table = by.tables[layer];
    int* counts = shi;                  // E
    int* starts = shi + E;              // E + 1, in rows
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    if (logits) {                       // a step of few tokens: the choosing is done here too, a warp a token
        for (int t = threadIdx.x >> 5; t < n / top; t += blockDim.x >> 5)
            route_token(logits + (size_t)t * ro.ld, E, top, ro, ids + (size_t)t * top, wts + (size_t)t * top,
                        threadIdx.x & 31);
        __syncthreads();
    }
    if (table) {                        // no router: a token's experts are its id's row of the table
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
            const int tok = by.token_ids[i / top];
            const bool known = tok >= 0 && tok < by.rows;
            if (!known) lsb_set_status(LSB_BAD_TOKEN);
            ids[i] = known ? table[(size_t)tok * top + i % top] : -1;
            wts[i] = by.weight;
        }
        __syncthreads();
    }
    for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0;
    for (int i = threadIdx.x; i < cap_tiles * tile; i += blockDim.x) { row_token[i] = -1; row_scale[i] = 0.f; }
    for (int i = threadIdx.x; i < cap_tiles; i += blockDim.x) tile_expert[i] = -1;
    __syncthreads();
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const int e = ids[i];
        if (e < 0 || e >= E) { lsb_set_status(LSB_BAD_ROW); pos[i] = -1; continue; }
        pos[i] = atomicAdd(&counts[e], 1);
    }
    __syncthreads();
    if (threadIdx.x < 32) {                 // running sum over the experts, a warp's width at a time
        const int lane = threadIdx.x;
        int at = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int n_rows = e0 + lane < E ? (counts[e0 + lane] + tile - 1) / tile * tile : 0;
            int sum = n_rows;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int below = __shfl_up_sync(0xffffffffu, sum, o);
                if (lane >= o) sum += below;
            }
            if (e0 + lane < E) starts[e0 + lane] = at + sum - n_rows;
            at += __shfl_sync(0xffffffffu, sum, 31);
        }
        if (lane == 0) starts[E] = at;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < E; e += blockDim.x)
        for (int ti = starts[e] / tile; ti < starts[e + 1] / tile && ti < cap_tiles; ++ti)
            tile_expert[ti] = e;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        if (pos[i] < 0) continue;
        const int p = starts[ids[i]] + pos[i];
        pos[i] = p;
        if (p < cap_tiles * tile) { row_token[p] = i / top; row_scale[p] = wts[i]; }
    }
}

// MODE 0 (up):   A row = T(scale * x[row_token]) (scale 1 unless on_input), B = w[e] [2F, K], gated
//                epilogue -> out T [capacity, F]
// MODE 2 (up, ungated): as MODE 0 with B = w[e] [N, K] and a plain activation -> out T [capacity, N]
// MODE 1 (down): A = h [capacity, K] T, B = w[e] [N, K] -> out 32-bit [capacity, N]
template <typename T, int MODE>
__global__ void __launch_bounds__(256)
moe_gemm_kernel(const T* __restrict__ A, const int* __restrict__ row_token,
                const float* __restrict__ row_scale, int on_input, const T* __restrict__ W,
                const int* __restrict__ tile_expert, void* __restrict__ out_, int N, int K, int act, float limit) {
    __shared__ float As[kTile][kTile + 1];
    __shared__ float Bs[kTile][kTile + 1];
    __shared__ int tok_sh[kTile];
    __shared__ float scale_sh[kTile];
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int e = tile_expert[blockIdx.y];
    if (e < 0) return;
    const int m0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
    const int tx = threadIdx.x % 32, ty = threadIdx.x / 32;
    if (threadIdx.x < kTile) {
        tok_sh[threadIdx.x] = row_token[m0 + threadIdx.x];
        scale_sh[threadIdx.x] = on_input ? row_scale[m0 + threadIdx.x] : 1.f;
    }
    __syncthreads();
    const T* B = W + (size_t)e * N * K;
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    for (int k0 = 0; k0 < K; k0 += kTile) {
        for (int i = ty; i < kTile; i += 8) {
            const int k = k0 + tx, n = n0 + i;
            float a = 0.f;
            if (k < K && tok_sh[i] >= 0) {
                if (MODE != 1)
                    a = lsb_to_float(lsb_from_float<T>(scale_sh[i] * lsb_to_float(A[(size_t)tok_sh[i] * K + k])));
                else
                    a = lsb_to_float(A[(size_t)(m0 + i) * K + k]);
            }
            As[i][tx] = a;
            Bs[i][tx] = (n < N && k < K) ? lsb_to_float(B[(size_t)n * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < kTile; ++k) {
            const float bv = Bs[tx][k];
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[j] += As[ty + 8 * j][k] * bv;
        }
        __syncthreads();
    }
    const int n = n0 + tx;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        const int m = m0 + ty + 8 * j;
        if (MODE == 0) {
            const float up = __shfl_down_sync(0xffffffffu, acc[j], 1);
            if (!(tx & 1) && n + 1 < N)
                ((T*)out_)[(size_t)m * (N / 2) + n / 2] = lsb_from_float<T>(moe_gate_mul(acc[j], up, act, limit));
        } else if (MODE == 2) {
            if (n < N) ((T*)out_)[(size_t)m * N + n] = lsb_from_float<T>(moe_plain(acc[j], act));
        } else if (n < N) {
            ((float*)out_)[(size_t)m * N + n] = acc[j];
        }
    }
}

// One block per (token, choice) pair: only rows that stand for a pair are written.  The padding
// rows of a tile keep whatever the buffer held: a row of a product depends on its own operand row
// alone, and nothing reads the padding rows' results.
template <typename T>
__global__ void moe_gather_kernel(const T* __restrict__ x, const int* __restrict__ pos,
                                  const float* __restrict__ wts, int on_input, int top, int capacity, int n,
                                  T* __restrict__ rows) {
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const size_t pair = blockIdx.x;
    const int r = pos[pair];
    if (r < 0 || r >= capacity) return;
    const size_t tok = pair / top;
    const float sc = on_input ? wts[pair] : 1.f;
    const T* src = x + tok * n;
    T* dst = rows + (size_t)r * n;
    if (sizeof(T) == 2 && n % 8 == 0 && (((uintptr_t)x | (uintptr_t)rows) & 15) == 0) {
        for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {      // 16 bytes a thread and pass
            uint4 raw = *reinterpret_cast<const uint4*>(src + i);
            __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const float2 f = __bfloat1622float2(p[k]);
                p[k] = __floats2bfloat162_rn(sc * f.x, sc * f.y);
            }
            *reinterpret_cast<uint4*>(dst + i) = raw;
        }
        return;
    }
    for (int i = threadIdx.x; i < n; i += blockDim.x)
        dst[i] = lsb_from_float<T>(sc * lsb_to_float(src[i]));
}

template <typename T, typename TY>
__global__ void moe_combine_kernel(const TY* __restrict__ y, const int* __restrict__ pos,
                                   const float* __restrict__ wts, int on_output, int top, int n,
                                   int capacity, T* __restrict__ out, const T* __restrict__ add,
                                   const float* __restrict__ add_gate, int gate_ld) {
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const size_t t = blockIdx.x;
    const float ag = add_gate ? 1.f / (1.f + expf(-add_gate[t * gate_ld])) : 1.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        float s = 0.f;
        for (int k = 0; k < top; ++k) {
            const int p = pos[t * top + k];
            if (p < 0 || p >= capacity) continue;
            const float v = lsb_to_float(y[(size_t)p * n + i]);
            s += on_output ? wts[t * top + k] * v : v;
        }
        if (add) s += ag * lsb_to_float(add[t * n + i]);          // (what every token passes besides its chosen experts)
        out[t * n + i] = lsb_from_float<T>(s);
    }
}

// The same for bfloat16 rows of a multiple of 8 columns: 16 bytes a thread, a token's choices eight at a time with
// all their rows in flight.
__global__ void __launch_bounds__(256)
moe_combine_vec_kernel(const __nv_bfloat16* __restrict__ y, const int* __restrict__ pos, const float* __restrict__ wts,
                       int on_output, int top, int n, int capacity, __nv_bfloat16* __restrict__ out,
                       const __nv_bfloat16* __restrict__ add, const float* __restrict__ add_gate, int gate_ld) {
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const size_t t = blockIdx.x;
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * 8;
    if (c >= n) return;
    float s[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    auto join = [&](const uint4& raw, float w) {
        const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const float2 f = __bfloat1622float2(p[j]);
            s[2 * j] += w * f.x;
            s[2 * j + 1] += w * f.y;
        }
    };
    uint4 shared_row = make_uint4(0u, 0u, 0u, 0u);
    float ag = 1.f;
    if (add) {
        shared_row = *reinterpret_cast<const uint4*>(add + t * n + c);
        if (add_gate) ag = add_gate[t * gate_ld];
    }
    for (int k0 = 0; k0 < top; k0 += 8) {
        uint4 rows[8];
        float w[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            rows[k] = make_uint4(0u, 0u, 0u, 0u);
            w[k] = 0.f;
            if (k0 + k < top) {
                const int p = pos[t * top + k0 + k];
                if (p >= 0 && p < capacity) {
                    rows[k] = *reinterpret_cast<const uint4*>(y + (size_t)p * n + c);
                    w[k] = on_output ? wts[t * top + k0 + k] : 1.f;
                }
            }
        }
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (k0 + k < top) join(rows[k], w[k]);
    }
    if (add) join(shared_row, add_gate ? 1.f / (1.f + expf(-ag)) : 1.f);
    __nv_bfloat162 o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = __floats2bfloat162_rn(s[2 * j], s[2 * j + 1]);
    *reinterpret_cast<uint4*>(out + t * n + c) = *reinterpret_cast<const uint4*>(o);
}

LSB_API int lsb_moe_tile() { return kTile; }

LSB_API int lsb_moe_route(const float* logits, int ld, int n_tokens, int E, int top, int score, int renorm,
                          const float* bias, int joins, float scale, float eps, int* ids, float* wts, cudaStream_t stream) {
    const RouteOpts ro = {score, renorm, bias, scale, eps, joins, ld};
    if (n_tokens <= 0) return 0;
    if (E <= 0 || top <= 0 || top > E || top > kMaxTop || score < 0 || score > 2 || ld < E) return (int)cudaErrorInvalidValue;
    const int warps_per_block = 4;
    return lsb_launch(moe_route_kernel, dim3((n_tokens + warps_per_block - 1) / warps_per_block),
                      dim3(32 * warps_per_block), 0, stream, 1, logits, n_tokens, E, top, ro, ids, wts);
}

// logits given (32-bit [tokens, E]): ids and wts are chosen here first (see lsb_moe_route) and written
LSB_API int lsb_moe_align(int* ids, float* wts, int n_tokens, int top, int E, int cap_tiles,
                          int tile, int* pos, int* row_token, float* row_scale, int* tile_expert,
                          const float* logits, int ld, int score, int renorm, const float* bias, int joins, float scale, float eps,
                          cudaStream_t stream) {
    const RouteOpts ro = {score, renorm, bias, scale, eps, joins, ld};
    const TokenRows by = {};
    if (n_tokens <= 0) return 0;
    const long long n = (long long)n_tokens * top;
    if (E <= 0 || E > 8192 || tile <= 0 || cap_tiles < (n + tile - 1) / tile + E) return (int)cudaErrorInvalidValue;
    if (logits && (top > kMaxTop || top > E || score < 0 || score > 2 || ld < E)) return (int)cudaErrorInvalidValue;
    return lsb_launch(moe_align_kernel, dim3(1), dim3(1024), (size_t)(2 * E + 1) * sizeof(int), stream, 1,
                      ids, wts, (int)n, top, E, cap_tiles, tile, pos, row_token, row_scale, tile_expert, logits, ro, by);
}

LSB_API int lsb_moe_max_tables() { return kMaxTables; }

// The same for `layers` layers whose experts are named by tables [table_rows, top] of the tokens' ids, each choice with
// the weight `weight`: every output has a leading dimension of `layers`.
LSB_API int lsb_moe_align_tables(const int* const* tables, int layers, const int* token_ids, int table_rows, float weight, int* ids,
                                 float* wts, int n_tokens, int top, int E, int cap_tiles, int tile, int* pos, int* row_token,
                                 float* row_scale, int* tile_expert, cudaStream_t stream) {
    if (n_tokens <= 0 || layers <= 0) return 0;
    const long long n = (long long)n_tokens * top;
    if (layers > kMaxTables || table_rows <= 0 || top <= 0 || E <= 0 || E > 8192 || tile <= 0 || n > 0x7fffffffLL ||
        cap_tiles < (n + tile - 1) / tile + E)
        return (int)cudaErrorInvalidValue;
    TokenRows by = {};
    for (int i = 0; i < layers; ++i) by.tables[i] = tables[i];
    by.token_ids = token_ids;
    by.rows = table_rows;
    by.weight = weight;
    const RouteOpts ro = {};
    return lsb_launch(moe_align_kernel, dim3(layers), dim3(1024), (size_t)(2 * E + 1) * sizeof(int), stream, 1, ids, wts, (int)n, top, E,
                      cap_tiles, tile, pos, row_token, row_scale, tile_expert, (const float*)nullptr, ro, by);
}

// rows[pos[t, k]] = T(wts[t, k] * x[t]): the operand of the grouped tensor-core product, which wants
// its rows in place
LSB_API int lsb_moe_gather(const void* x, int dtype, const int* pos, const float* wts, int on_input,
                           int n_tokens, int top, int capacity, int n, void* rows, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    LSB_DISPATCH_DTYPE(dtype, return lsb_launch(moe_gather_kernel<T>, dim3((unsigned)((long long)n_tokens * top)), dim3(128),
                                                0, stream, 1, (const T*)x, pos, wts, on_input, top, capacity, n,
                                                (T*)rows));
    return 0;
}

// `plain`: w is [E, F, K] and act a plain activation; else [E, 2F, K], gate and up rows alternating
LSB_API int lsb_moe_up(const void* x, int dtype, const int* row_token, const float* row_scale, int on_input,
                       const void* w, const int* tile_expert, int cap_tiles, void* out, int F, int K,
                       int act, float limit, int plain, cudaStream_t stream) {
    if (cap_tiles <= 0) return 0;
    if (F <= 0 || K <= 0 || cap_tiles > 65535) return (int)cudaErrorInvalidValue;
    dim3 grid(((plain ? F : 2 * F) + kTile - 1) / kTile, cap_tiles);
    if (plain)
        LSB_DISPATCH_DTYPE(dtype, return lsb_launch(moe_gemm_kernel<T, 2>, grid, dim3(256), 0, stream, 1,
                                                    (const T*)x, row_token, row_scale, on_input, (const T*)w,
                                                    tile_expert, out, F, K, act, limit));
    LSB_DISPATCH_DTYPE(dtype, return lsb_launch(moe_gemm_kernel<T, 0>, grid, dim3(256), 0, stream, 1,
                                                (const T*)x, row_token, row_scale, on_input, (const T*)w,
                                                tile_expert, out, 2 * F, K, act, limit));
    return 0;
}

LSB_API int lsb_moe_down(const void* h, int dtype, const int* row_token, const void* w,
                         const int* tile_expert, int cap_tiles, float* out, int N, int K,
                         cudaStream_t stream) {
    if (cap_tiles <= 0) return 0;
    if (N <= 0 || K <= 0 || cap_tiles > 65535) return (int)cudaErrorInvalidValue;
    dim3 grid((N + kTile - 1) / kTile, cap_tiles);
    LSB_DISPATCH_DTYPE(dtype, return lsb_launch(moe_gemm_kernel<T, 1>, grid, dim3(256), 0, stream, 1,
                                                (const T*)h, row_token, (const float*)nullptr, 0, (const T*)w,
                                                tile_expert, (void*)out, N, K, 0, 0.f));
    return 0;
}

// y_same: the expert rows are stored in the output's type (the tensor-core path), else 32-bit
LSB_API int lsb_moe_combine(const void* y, int y_same, const int* pos, const float* wts, int on_output,
                            int n_tokens, int top, int n, int capacity, void* out, int dtype, const void* add,
                            const float* add_gate, int gate_ld, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (dtype == LSB_BF16 && y_same && n % 8 == 0 &&
        (((uintptr_t)y | (uintptr_t)out | (uintptr_t)add) & 15) == 0) {
        const int chunks = n / 8, threads = chunks >= 256 ? 256 : (chunks + 31) / 32 * 32;
        return lsb_launch(moe_combine_vec_kernel, dim3(n_tokens, (chunks + threads - 1) / threads), dim3(threads), 0, stream, 1,
                          (const __nv_bfloat16*)y, pos, wts, on_output, top, n, capacity, (__nv_bfloat16*)out,
                          (const __nv_bfloat16*)add, add_gate, gate_ld);
    }
    LSB_DISPATCH_DTYPE(dtype, {
        if (y_same)
            return lsb_launch(moe_combine_kernel<T, T>, dim3(n_tokens), dim3(256), 0, stream, 1, (const T*)y, pos,
                              wts, on_output, top, n, capacity, (T*)out, (const T*)add, add_gate, gate_ld);
        return lsb_launch(moe_combine_kernel<T, float>, dim3(n_tokens), dim3(256), 0, stream, 1, (const float*)y,
                          pos, wts, on_output, top, n, capacity, (T*)out, (const T*)add, add_gate, gate_ld);
    });
    return 0;
}
