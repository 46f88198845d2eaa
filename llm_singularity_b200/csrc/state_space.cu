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
// kernel, which runs when every token has been prepared.  All of it is 32-bit; u is rounded to the
// compute dtype where that is bfloat16.
#include "common.cuh"

LSB_DEFINE_STATUS()

constexpr int kPrepThreads = 128;
constexpr int kPrepTokens = 16;          // tokens a thread takes of its channel, one after another

__device__ __forceinline__ float ss_silu(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float ss_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct PrepArgs {
    const float* proj; long long ld; int x_off, dt_off;       // x | B | C side by side from x_off on
    int channels, heads, taps, tokens;
    const float *conv, *conv_bias, *dt_bias, *a_log;            // conv [channels, taps]
    float* conv_state; int n_slots;                             // [slots, taps - 1, channels]
    const int *token_req, *q_start, *table_rows;
    float *keep, *write, *log_keep;                             // [tokens, heads]
    int update_state;
};

// W channels a thread (1 or 4), TAPS 2 .. 4 (the inputs of earlier tokens in registers) or 0 (any number).
template <typename T, int W, int TAPS>
__global__ void __launch_bounds__(kPrepThreads) state_space_prep_kernel(PrepArgs a, T* __restrict__ u) {
    lsb_pdl_launch_dependents();
    const int first = blockIdx.y * kPrepTokens, last = min(first + kPrepTokens, a.tokens);
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
        if (W == 4) {
            const float4 x = *reinterpret_cast<const float4*>(p);
            v[0] = x.x; v[W > 1 ? 1 : 0] = x.y; v[W > 2 ? 2 : 0] = x.z; v[W > 3 ? 3 : 0] = x.w;
        } else {
            v[0] = p[0];
        }
    };
    int r = -1, t0 = 0, slot = 0;
    for (int t = first; t < last; ++t) {
        const int rt = a.token_req[t];
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
        load(a.proj + (size_t)t * a.ld + a.x_off + c0, now);
#pragma unroll
        for (int w = 0; w < W; ++w) acc[w] = bias[w];
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
        if (W == 4) {
            if constexpr (sizeof(T) == 2) {
                const __nv_bfloat162 p = __floats2bfloat162_rn(ss_silu(acc[0]), ss_silu(acc[W > 1 ? 1 : 0]));
                const __nv_bfloat162 q = __floats2bfloat162_rn(ss_silu(acc[W > 2 ? 2 : 0]), ss_silu(acc[W > 3 ? 3 : 0]));
                *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&p), *reinterpret_cast<const uint32_t*>(&q));
            } else {
                *reinterpret_cast<float4*>(dst) = make_float4(ss_silu(acc[0]), ss_silu(acc[W > 1 ? 1 : 0]), ss_silu(acc[W > 2 ? 2 : 0]),
                                                              ss_silu(acc[W > 3 ? 3 : 0]));
            }
        } else {
            dst[0] = lsb_from_float<T>(ss_silu(acc[0]));
        }
    }
}

struct OutArgs {
    const float* y;                                             // [tokens, heads * V], the walk's read-out
    const float* proj; long long ld; int x_off;                 // z in the first heads * V columns
    const float *d, *w;                                         // [heads], [heads * V]
    int heads, V, groups; float eps;
    int channels, taps;                                         // the convolution's state (taps 0: not updated here)
    float* conv_state; int n_slots;
    const int *token_req, *q_start, *table_rows;
};

// block (token, norm group); with taps > 1 one block more per token, which in a request's last token
// replaces the request's convolution inputs
template <typename T, int W>
__global__ void __launch_bounds__(256) state_space_output_kernel(OutArgs a, const T* __restrict__ u, T* __restrict__ out) {
    extern __shared__ float v_sh[];
    __shared__ float scratch[33];
    lsb_pdl_launch_dependents();
    const size_t t = blockIdx.x;
    const int inner = a.heads * a.V, gs = inner / a.groups;
    if ((int)blockIdx.y == a.groups) {
        lsb_pdl_wait();
        const int r = a.token_req[t], t0 = a.q_start[r], n = a.q_start[r + 1] - t0, m = a.taps - 1;
        if ((int)t != t0 + n - 1) return;
        const int slot = a.table_rows[r];
        if (slot < 0 || slot >= a.n_slots) {
            if (threadIdx.x == 0) lsb_set_status(LSB_BAD_ROW);
            return;
        }
        for (int c = threadIdx.x; c < a.channels; c += blockDim.x) {
            float* s = a.conv_state + (size_t)slot * m * a.channels + c;
            for (int j = 0; j < m; ++j) {                       // in order: row j may take what row j + n held
                const int back = m - 1 - j;                     // tokens before the last one
                s[(size_t)j * a.channels] = back < n ? a.proj[((size_t)t - back) * a.ld + a.x_off + c] : s[(size_t)(j + n) * a.channels];
            }
        }
        return;
    }
    const int base = blockIdx.y * gs;
    lsb_pdl_wait();
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < gs; i += blockDim.x * W) {
        const int c = base + i;
        float y[W], z[W], x[W];
        if (W == 4) {
            const float4 yv = *reinterpret_cast<const float4*>(a.y + t * inner + c), zv = *reinterpret_cast<const float4*>(a.proj + t * a.ld + c);
            y[0] = yv.x; y[W > 1 ? 1 : 0] = yv.y; y[W > 2 ? 2 : 0] = yv.z; y[W > 3 ? 3 : 0] = yv.w;
            z[0] = zv.x; z[W > 1 ? 1 : 0] = zv.y; z[W > 2 ? 2 : 0] = zv.z; z[W > 3 ? 3 : 0] = zv.w;
        } else {
            y[0] = a.y[t * inner + c];
            z[0] = a.proj[t * a.ld + c];
        }
#pragma unroll
        for (int w = 0; w < W; ++w) x[w] = lsb_to_float(u[t * a.channels + c + w]);
#pragma unroll
        for (int w = 0; w < W; ++w) {
            const float v = (y[w] + a.d[(c + w) / a.V] * x[w]) * ss_silu(z[w]);
            v_sh[i + w] = v;
            ss += v * v;
        }
    }
    const float inv = rsqrtf(lsb_block_sum(ss, scratch) / (float)gs + a.eps);
    for (int i = threadIdx.x * W; i < gs; i += blockDim.x * W) {
        const int c = base + i;
        T o[W];
#pragma unroll
        for (int w = 0; w < W; ++w) o[w] = lsb_from_float<T>(v_sh[i + w] * inv * a.w[c + w]);
        if (W == 4) {
            if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(out + t * inner + c) = *reinterpret_cast<const uint2*>(o);
            else *reinterpret_cast<float4*>(out + t * inner + c) = make_float4(o[0], o[W > 1 ? 1 : 0], o[W > 2 ? 2 : 0], o[W > 3 ? 3 : 0]);
        } else {
            out[t * inner + c] = o[0];
        }
    }
}

// proj: 32-bit rows `ld` apart; x | B | C in `channels` columns from x_off on, dt's projection in `heads` columns
// from dt_off on.  u [tokens, channels] in `dtype`.  update_state: every request of the step brings one token,
// and its convolution inputs are replaced here.
LSB_API int lsb_state_space_prep(const float* proj, long long ld, int x_off, int dt_off, int tokens, int channels, int heads, int taps,
                                 const float* conv, const float* conv_bias, const float* dt_bias, const float* a_log,
                                 float* conv_state, int n_slots, const int* token_req, const int* q_start, const int* table_rows,
                                 void* u, int dtype, float* keep, float* write, float* log_keep, int update_state,
                                 cudaStream_t stream) {
    if (tokens <= 0) return 0;
    if (channels <= 0 || heads <= 0 || taps < 1 || (taps > 1 && !conv_state)) return (int)cudaErrorInvalidValue;
    PrepArgs a;
    a.proj = proj; a.ld = ld; a.x_off = x_off; a.dt_off = dt_off;
    a.channels = channels; a.heads = heads; a.taps = taps; a.tokens = tokens;
    a.conv = conv; a.conv_bias = conv_bias; a.dt_bias = dt_bias; a.a_log = a_log;
    a.conv_state = conv_state; a.n_slots = n_slots;
    a.token_req = token_req; a.q_start = q_start; a.table_rows = table_rows;
    a.keep = keep; a.write = write; a.log_keep = log_keep;
    a.update_state = update_state;
    const bool vec = (uintptr_t)proj % 16 == 0 && (uintptr_t)u % 16 == 0 && (uintptr_t)conv_state % 16 == 0 && ld % 4 == 0 &&
                     x_off % 4 == 0 && channels % 4 == 0;
    const int per_block = kPrepThreads * (vec ? 4 : 1);
    const long long tiles = (tokens + kPrepTokens - 1) / kPrepTokens;
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
LSB_API int lsb_state_space_output(const float* y, const float* proj, long long ld, int x_off, const void* u, int channels,
                                   const float* d, const float* w, int tokens, int heads, int V, int groups, float eps, int taps,
                                   float* conv_state, int n_slots, const int* token_req, const int* q_start, const int* table_rows,
                                   void* out, int dtype, cudaStream_t stream) {
    if (tokens <= 0) return 0;
    const int inner = heads * V;
    if (heads <= 0 || V <= 0 || groups <= 0 || inner % groups || channels < inner || groups >= 65535) return (int)cudaErrorInvalidValue;
    OutArgs a;
    a.y = y; a.proj = proj; a.ld = ld; a.x_off = x_off;
    a.d = d; a.w = w; a.heads = heads; a.V = V; a.groups = groups; a.eps = eps;
    a.channels = channels; a.taps = taps; a.conv_state = conv_state; a.n_slots = n_slots;
    a.token_req = token_req; a.q_start = q_start; a.table_rows = table_rows;
    const int gs = inner / groups;
    const size_t smem = (size_t)gs * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const bool vec = (uintptr_t)y % 16 == 0 && (uintptr_t)proj % 16 == 0 && (uintptr_t)out % 16 == 0 && ld % 4 == 0 && gs % 4 == 0;
    int threads = ((gs / (vec ? 4 : 1) + 31) / 32) * 32;
    threads = threads < 32 ? 32 : threads > 256 ? 256 : threads;
    dim3 grid(tokens, groups + (taps > 1 ? 1 : 0));
#define LSB_SS_OUT(W)                                                                                              \
    do {                                                                                                           \
        if (smem > 48 * 1024) {                                                                                    \
            int rc = (int)cudaFuncSetAttribute(state_space_output_kernel<T, W>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (rc) return rc;                                                                                     \
        }                                                                                                          \
        return lsb_launch(state_space_output_kernel<T, W>, grid, dim3(threads), smem, stream, 1, a, (const T*)u, (T*)out); \
    } while (0)
    LSB_DISPATCH_DTYPE(dtype, {
        if (vec) LSB_SS_OUT(4);
        else LSB_SS_OUT(1);
    });
#undef LSB_SS_OUT
    return 0;
}
