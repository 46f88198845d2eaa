// Around the walk of a state-space memory (S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x): what
// enters it and what becomes of its read-out.
//
//   state_space_prep    per token, from the 32-bit rows of the wide projection: a causal convolution per
//                       channel over time (x, B and C together) with a bias, then silu -> u; and per head
//                       dt = softplus(. + dt_bias), the fade exp(-exp(A_log) dt) and its logarithm.
//   state_space_output  v = (y + D x) * silu(z); v / sqrt(mean over its norm group of v^2 + eps) * w.
//
// The last taps - 1 inputs of the convolution are state, one row per request slot.  They are read by
// the preparation for a portion's first tokens and replaced for the next step: by the preparation itself
// where every request brings one token (a thread then owns a request's channel), else by the output
// kernel, which runs when every token has been prepared.  All arithmetic is 32-bit; u is rounded to the
// compute dtype where that is bfloat16.
#include "common.cuh"

LSB_DEFINE_STATUS()

constexpr int kPrepThreads = 128;
constexpr int kPrepTokens = 16;          // tokens a thread takes of its channel, one after another (one where a step has few)

// z / (1 + e^-z).  Where the result is rounded to bfloat16 the special-function unit's exponential and an
// approximate division (each good to about 1e-7 relative) cost a quarter of the exact ones.
template <typename T>
__device__ __forceinline__ float ss_silu(float z) {
    if constexpr (sizeof(T) == 2) return __fdividef(z, 1.f + __expf(-z));
    else return z / (1.f + expf(-z));
}
__device__ __forceinline__ float ss_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct PrepArgs {
    const float* proj; long long ld; int x_off, dt_off;         // x | B | C side by side from x_off on; dt, a column a head
    int channels, heads, taps, tokens, tile;
    const float *conv, *conv_bias, *dt_bias, *a_log;            // conv [channels, taps]
    float* conv_state; int n_slots;                             // [slots, taps - 1, channels]
    const int *token_req, *q_start, *table_rows;
    float *keep, *write, *log_keep;                             // [tokens, heads]
    int update_state;
};

// four consecutive elements as floats, and back
__device__ __forceinline__ float4 ss_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ss_load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void ss_store4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void ss_store4(__nv_bfloat16* p, float a, float b, float c, float d) {
    const __nv_bfloat162 u = __floats2bfloat162_rn(a, b), v = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&u), *reinterpret_cast<const uint32_t*>(&v));
}

// W channels a thread (1 or 4), TAPS 2 .. 4 (the inputs of earlier tokens in registers) or 0 (any number).
template <typename T, int W, int TAPS>
__global__ void __launch_bounds__(kPrepThreads) state_space_prep_kernel(PrepArgs a, T* __restrict__ u) {
    lsb_pdl_launch_dependents();
    const int first = blockIdx.y * a.tile, last = min(first + a.tile, a.tokens);
    const int taps = TAPS ? TAPS : a.taps, m = taps - 1;
    if (blockIdx.x == gridDim.x - 1) {                          // the heads' step sizes and fades
        lsb_pdl_wait();
        for (int w = threadIdx.x; w < (last - first) * a.heads; w += kPrepThreads) {
            const int t = first + w / a.heads, h = w % a.heads;
            const float dt = ss_softplus(a.proj[(size_t)t * a.ld + a.dt_off + h] + a.dt_bias[h]);
            const float lk = -expf(a.a_log[h]) * dt;
            const size_t at = (size_t)t * a.heads + h;
            a.write[at] = dt;
            a.log_keep[at] = lk;
            a.keep[at] = expf(lk);
        }
        return;
    }
    const int c0 = (blockIdx.x * kPrepThreads + threadIdx.x) * W;
    if (c0 >= a.channels) return;
    constexpr int HR = TAPS > 1 ? TAPS - 1 : 1;
    float taps_r[TAPS ? TAPS : 1][W], bias[W], hist[HR][W];
#pragma unroll
    for (int w = 0; w < W; ++w) {
        bias[w] = a.conv_bias[c0 + w];
        if (TAPS) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j) taps_r[j][w] = a.conv[(size_t)(c0 + w) * TAPS + j];
        }
    }
    lsb_pdl_wait();
    auto load = [&](const float* p, float (&v)[W]) {
        if constexpr (W == 4) {
            const float4 x = ss_load4(p);
            v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
        } else {
            v[0] = p[0];
        }
    };
    int r = -1, t0 = 0, slot = 0;
    constexpr int AHEAD = 8;
    for (int t8 = first; t8 < last; t8 += AHEAD) {             // eight tokens' inputs in flight together
    float now8[AHEAD][W];
    int req8[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
        if (t8 + k < last) {
            req8[k] = a.token_req[t8 + k];
            load(a.proj + (size_t)(t8 + k) * a.ld + a.x_off + c0, now8[k]);
        }
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
        const int t = t8 + k;
        if (t >= last) break;
        const int rt = req8[k];
        const bool fresh = rt != r;                             // a request's first token here
        if (fresh) {
            r = rt;
            t0 = a.q_start[r];
            slot = a.table_rows[r];
        }
        if (slot < 0 || slot >= a.n_slots) {
            lsb_set_status(LSB_BAD_ROW);
            continue;
        }
        const float* old = a.conv_state + (size_t)slot * m * a.channels + c0;
        // the input `back` tokens before t, from this portion or from the state
        auto earlier = [&](int back, float (&v)[W]) {
            const int at = t - back;
            if (at >= t0) load(a.proj + (size_t)at * a.ld + a.x_off + c0, v);
            else load(old + (size_t)(at - t0 + m) * a.channels, v);
        };
        float now[W], acc[W];
#pragma unroll
        for (int w = 0; w < W; ++w) {
            now[w] = now8[k][w];
            acc[w] = bias[w];
        }
        if (TAPS) {
            if (fresh) {
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) earlier(TAPS - 1 - j, hist[j]);
            }
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) {
#pragma unroll
                for (int w = 0; w < W; ++w) acc[w] += taps_r[j][w] * hist[j][w];
            }
#pragma unroll
            for (int w = 0; w < W; ++w) acc[w] += taps_r[TAPS ? TAPS - 1 : 0][w] * now[w];
            if (a.update_state) {                               // (one token a request: hist is what the state held)
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
#pragma unroll
                    for (int w = 0; w < W; ++w)
                        a.conv_state[((size_t)slot * m + j) * a.channels + c0 + w] = j + 1 < TAPS - 1 ? hist[j + 1 < HR ? j + 1 : 0][w] : now[w];
                }
            }
#pragma unroll
            for (int j = 0; j + 1 < TAPS - 1; ++j) {
#pragma unroll
                for (int w = 0; w < W; ++w) hist[j][w] = hist[j + 1 < HR ? j + 1 : 0][w];
            }
            if (TAPS > 1) {
#pragma unroll
                for (int w = 0; w < W; ++w) hist[TAPS > 1 ? TAPS - 2 : 0][w] = now[w];
            }
        } else {
            float v[W];
            for (int j = 0; j < taps; ++j) {
                earlier(m - j, v);
#pragma unroll
                for (int w = 0; w < W; ++w) acc[w] += a.conv[(size_t)(c0 + w) * taps + j] * v[w];
            }
            if (a.update_state) {
                for (int j = 0; j < m; ++j) {                   // (row j takes what row j + 1 held: in order, one thread)
                    earlier(m - 1 - j, v);
#pragma unroll
                    for (int w = 0; w < W; ++w) a.conv_state[((size_t)slot * m + j) * a.channels + c0 + w] = v[w];
                }
            }
        }
        T* dst = u + (size_t)t * a.channels + c0;
        if constexpr (W == 4) {
            ss_store4(dst, ss_silu<T>(acc[0]), ss_silu<T>(acc[1]), ss_silu<T>(acc[2]), ss_silu<T>(acc[3]));
        } else {
            dst[0] = lsb_from_float<T>(ss_silu<T>(acc[0]));
        }
    }
    }
}

struct OutArgs {
    const float* y;                                             // [tokens, heads * V], the walk's read-out
    const float* proj; long long ld; int x_off;                // z in the first heads * V columns
    const float *d, *w;                                         // [heads * V] each (d the same for a head's channels)
    int heads, V, groups; float eps;
    int channels, taps;                                         // the convolution's state (taps 0: not updated here)
    float* conv_state; int n_slots;
    const int *token_req, *q_start, *table_rows;
};

// A request's convolution inputs for the next step: its last taps - 1, from the portion and what the state held.
__device__ __forceinline__ void keep_inputs(const OutArgs& a, size_t t) {
    const int r = a.token_req[t], t0 = a.q_start[r], n = a.q_start[r + 1] - t0, m = a.taps - 1;
    if ((int)t != t0 + n - 1) return;
    const int slot = a.table_rows[r];
    if (slot < 0 || slot >= a.n_slots) {
        if (threadIdx.x == 0) lsb_set_status(LSB_BAD_ROW);
        return;
    }
    for (int c = threadIdx.x; c < a.channels; c += blockDim.x) {
        float* s = a.conv_state + (size_t)slot * m * a.channels + c;
        for (int j = 0; j < m; ++j) {                           // in order: row j may take what row j + n held
            const int back = m - 1 - j;                         // tokens before the last one
            s[(size_t)j * a.channels] = back < n ? a.proj[((size_t)t - back) * a.ld + a.x_off + c] : s[(size_t)(j + n) * a.channels];
        }
    }
}

constexpr int kOutRegs = 2, kOutThreads = 512;

// Block (token, norm group); with taps > 1 one block more per token, which in a request's last token replaces
// the request's convolution inputs.  Four channels a thread and pass, a group of up to 4,096 channels in
// registers between the two passes.
template <typename T>
__global__ void __launch_bounds__(kOutThreads, 3) state_space_output_vec_kernel(OutArgs a, const T* __restrict__ u, T* __restrict__ out) {
    __shared__ float scratch[33];
    lsb_pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int inner = a.heads * a.V, gs = inner / a.groups;
    lsb_pdl_wait();
    if ((int)blockIdx.y == a.groups) {
        keep_inputs(a, t);
        return;
    }
    const int base = blockIdx.y * gs, step = blockDim.x * 4;
    const float* yr = a.y + t * inner + base;
    const float* zr = a.proj + t * a.ld + base;
    const T* xr = u + t * a.channels + base;
    float4 v[kOutRegs], z[kOutRegs], x[kOutRegs];
#pragma unroll
    for (int k = 0; k < kOutRegs; ++k) {
        const int i = threadIdx.x * 4 + k * step;
        v[k] = z[k] = x[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < gs) {
            v[k] = ss_load4(yr + i);
            z[k] = ss_load4(zr + i);
            x[k] = ss_load4(xr + i);
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < kOutRegs; ++k) {
        const int i = threadIdx.x * 4 + k * step;
        if (i < gs) {
            const float4 d = ss_load4(a.d + base + i);
            v[k].x = (v[k].x + d.x * x[k].x) * ss_silu<T>(z[k].x);
            v[k].y = (v[k].y + d.y * x[k].y) * ss_silu<T>(z[k].y);
            v[k].z = (v[k].z + d.z * x[k].z) * ss_silu<T>(z[k].z);
            v[k].w = (v[k].w + d.w * x[k].w) * ss_silu<T>(z[k].w);
            ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
        }
    }
    const float inv = rsqrtf(lsb_block_sum(ss, scratch) / (float)gs + a.eps);
#pragma unroll
    for (int k = 0; k < kOutRegs; ++k) {
        const int i = threadIdx.x * 4 + k * step;
        if (i < gs) {
            const float4 w = ss_load4(a.w + base + i);
            ss_store4(out + t * inner + base + i, v[k].x * inv * w.x, v[k].y * inv * w.y, v[k].z * inv * w.z, v[k].w * inv * w.w);
        }
    }
}

// The same for any sizes.
template <typename T>
__global__ void __launch_bounds__(256) state_space_output_kernel(OutArgs a, const T* __restrict__ u, T* __restrict__ out) {
    extern __shared__ float v_sh[];
    __shared__ float scratch[33];
    lsb_pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int inner = a.heads * a.V, gs = inner / a.groups;
    lsb_pdl_wait();
    if ((int)blockIdx.y == a.groups) {
        keep_inputs(a, t);
        return;
    }
    const int base = blockIdx.y * gs;
    float ss = 0.f;
    for (int i = threadIdx.x; i < gs; i += blockDim.x) {
        const int c = base + i;
        const float v = (a.y[t * inner + c] + a.d[c] * lsb_to_float(u[t * a.channels + c])) *
                        ss_silu<T>(a.proj[t * a.ld + c]);
        v_sh[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(lsb_block_sum(ss, scratch) / (float)gs + a.eps);
    for (int i = threadIdx.x; i < gs; i += blockDim.x) out[t * inner + base + i] = lsb_from_float<T>(v_sh[i] * inv * a.w[base + i]);
}

// proj: 32-bit rows `ld` apart; x | B | C in `channels` columns from x_off on, dt's projection in `heads` columns
// from dt_off on.  u [tokens, channels] in `dtype`.  update_state: every request of the step brings one token,
// and its convolution inputs are replaced here.
LSB_API int lsb_state_space_prep(const float* proj, long long ld, int x_off, int dt_off, int tokens, int channels, int heads, int taps, const float* conv, const float* conv_bias, const float* dt_bias,
                                 const float* a_log, float* conv_state, int n_slots, const int* token_req, const int* q_start,
                                 const int* table_rows, void* u, int dtype, float* keep, float* write, float* log_keep,
                                 int update_state, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (channels <= 0 || heads <= 0 || taps < 1 || (taps > 1 && !conv_state)) return (int)cudaErrorInvalidValue;
    PrepArgs a;
    a.proj = proj; a.ld = ld; a.x_off = x_off; a.dt_off = dt_off;
    a.channels = channels; a.heads = heads; a.taps = taps; a.tokens = tokens;
    a.tile = tokens <= 64 ? 1 : kPrepTokens;
    a.conv = conv; a.conv_bias = conv_bias; a.dt_bias = dt_bias; a.a_log = a_log;
    a.conv_state = conv_state; a.n_slots = n_slots;
    a.token_req = token_req; a.q_start = q_start; a.table_rows = table_rows;
    a.keep = keep; a.write = write; a.log_keep = log_keep;
    a.update_state = update_state;
    const bool vec = (uintptr_t)proj % 16 == 0 && (uintptr_t)u % 16 == 0 && (uintptr_t)conv_state % 16 == 0 && ld % 4 == 0 &&
                     x_off % 4 == 0 && channels % 4 == 0;
    const int per_block = kPrepThreads * (vec ? 4 : 1);
    const long long tiles = (tokens + a.tile - 1) / a.tile;
    if (tiles > 65535) return (int)cudaErrorInvalidValue;
    dim3 grid((channels + per_block - 1) / per_block + 1, (unsigned)tiles);
#define LSB_SS_PREP(W, TAPS) return lsb_launch(state_space_prep_kernel<T, W, TAPS>, grid, dim3(kPrepThreads), 0, stream, 1, a, (T*)u)
#define LSB_SS_PREP_TAPS(W)                   \
    do {                                      \
        if (taps == 4) LSB_SS_PREP(W, 4);     \
        else if (taps == 3) LSB_SS_PREP(W, 3); \
        else if (taps == 2) LSB_SS_PREP(W, 2); \
        else LSB_SS_PREP(W, 0);               \
    } while (0)
    LSB_DISPATCH_DTYPE(dtype, {
        if (vec) LSB_SS_PREP_TAPS(4);
        else LSB_SS_PREP_TAPS(1);
    });
#undef LSB_SS_PREP_TAPS
#undef LSB_SS_PREP
    return 0;
}

// taps <= 1: the convolution's state is left alone
LSB_API int lsb_state_space_output(const float* y, const float* proj, long long ld, int x_off, const void* u,
                                   int channels, const float* d, const float* w, int tokens, int heads, int V, int groups, float eps,
                                   int taps, float* conv_state, int n_slots, const int* token_req, const int* q_start,
                                   const int* table_rows, void* out, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    const int inner = heads * V;
    if (heads <= 0 || V <= 0 || groups <= 0 || inner % groups || channels < inner || groups >= 65535)
        return (int)cudaErrorInvalidValue;
    OutArgs a;
    a.y = y; a.proj = proj; a.ld = ld; a.x_off = x_off;
    a.d = d; a.w = w; a.heads = heads; a.V = V; a.groups = groups; a.eps = eps;
    a.channels = channels; a.taps = taps; a.conv_state = conv_state; a.n_slots = n_slots;
    a.token_req = token_req; a.q_start = q_start; a.table_rows = table_rows;
    const int gs = inner / groups;
    const size_t smem = (size_t)gs * sizeof(float);
    const bool vec = (uintptr_t)y % 16 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)u % 16 == 0 &&
                     (uintptr_t)w % 16 == 0 && ld % 4 == 0 && gs % 4 == 0 && (uintptr_t)d % 16 == 0 && channels % 4 == 0 && gs <= 4 * kOutThreads * kOutRegs;
    if (!vec && smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    int threads = ((gs / (vec ? 4 : 1) + 31) / 32) * 32;
    const int most = vec ? kOutThreads : 256;
    threads = threads < 32 ? 32 : threads > most ? most : threads;
    dim3 grid(tokens, groups + (taps > 1 ? 1 : 0));
    LSB_DISPATCH_DTYPE(dtype, {
        if (vec) return lsb_launch(state_space_output_vec_kernel<T>, grid, dim3(threads), 0, stream, 1, a, (const T*)u, (T*)out);
        if (smem > 48 * 1024) {
            int rc = (int)cudaFuncSetAttribute(state_space_output_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (rc) return rc;
        }
        return lsb_launch(state_space_output_kernel<T>, grid, dim3(threads), smem, stream, 1, a, (const T*)u, (T*)out);
    });
    return 0;
}
