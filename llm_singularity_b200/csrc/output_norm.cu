// The norm behind a sublayer and the sum into the stream, for arrangements whose sublayers read the
// stream itself:
//
//     x <- x + unit(v) * w        copy <- T(x)        unit(v) = v / sqrt(mean(v^2) + eps)
//
// where v is the sublayer's result, formed here in 32-bit from what the sublayer's last kernels left:
//
//   terms        v = sum_b s_b * y_b + bias     results of mixers side by side with their factors and the
//                                               biases of their output projections (or one result alone)
//   expert rows  v = sum_k wts[t, k] * y[pos[t, k]]     a token's chosen experts' rows, in their order
//
// One block per row.  A row's values wait in registers between the two passes (rows up to 4,096 wide
// in whole 16 bytes) or in shared memory (any width).  `copy` is the operand of the products that read
// the stream next; in 32-bit storage they read the stream itself and there is no copy.
#include "common.cuh"

LSB_DEFINE_STATUS()

constexpr int kJoinThreads = 256;
constexpr int kJoinRegs = 4;
constexpr int kMaxTerms = 4;

struct JoinArgs {
    float* x;
    const void* y[kMaxTerms];
    float s[kMaxTerms];
    int terms;
    const float* bias;
    const int* pos;             // expert rows: row of each (token, choice) in y[0]
    const float* wts;
    int top, capacity;
    const float* w;
    float eps;
    void* copy;
    int hidden;
};

__device__ __forceinline__ float4 join_load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 join_load4(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void join_store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void join_store4(__nv_bfloat16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
__device__ __forceinline__ void join_fma4(float4& a, float s, const float4& v) {
    a.x += s * v.x;
    a.y += s * v.y;
    a.z += s * v.z;
    a.w += s * v.w;
}

template <typename TY, typename T, bool EXPERTS>
__global__ void __launch_bounds__(kJoinThreads) join_norm_vec_kernel(JoinArgs a) {
    __shared__ float scratch[33];
    lsb_pdl_launch_dependents();
    const int hidden = a.hidden;
    const size_t t = blockIdx.x;
    float4 v[kJoinRegs], x[kJoinRegs];
    lsb_pdl_wait();
    float* xr = a.x + t * hidden;
#pragma unroll
    for (int u = 0; u < kJoinRegs; ++u) {
        const int i = 4 * (threadIdx.x + u * kJoinThreads);
        v[u] = x[u] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < hidden) {
            x[u] = join_load4(xr + i);
            if (a.bias) v[u] = join_load4(a.bias + i);
        }
    }
    if (EXPERTS) {
        const TY* y = (const TY*)a.y[0];
        for (int k0 = 0; k0 < a.top; k0 += 4) {                 // four rows in flight
            const TY* row[4];
            float s[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int p = k0 + k < a.top ? a.pos[t * a.top + k0 + k] : -1;
                const bool ok = p >= 0 && p < a.capacity;
                row[k] = ok ? y + (size_t)p * hidden : nullptr;
                s[k] = ok ? a.wts[t * a.top + k0 + k] : 0.f;
            }
#pragma unroll
            for (int u = 0; u < kJoinRegs; ++u) {
                const int i = 4 * (threadIdx.x + u * kJoinThreads);
                if (i < hidden) {
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (row[k]) join_fma4(v[u], s[k], join_load4(row[k] + i));
                }
            }
        }
    } else {
#pragma unroll
        for (int b = 0; b < kMaxTerms; ++b) {
            if (b < a.terms) {
                const TY* y = (const TY*)a.y[b] + t * hidden;
#pragma unroll
                for (int u = 0; u < kJoinRegs; ++u) {
                    const int i = 4 * (threadIdx.x + u * kJoinThreads);
                    if (i < hidden) join_fma4(v[u], a.s[b], join_load4(y + i));
                }
            }
        }
    }
    float ss = 0.f;
#pragma unroll
    for (int u = 0; u < kJoinRegs; ++u) ss += v[u].x * v[u].x + v[u].y * v[u].y + v[u].z * v[u].z + v[u].w * v[u].w;
    const float inv = rsqrtf(lsb_block_sum(ss, scratch) / (float)hidden + a.eps);
#pragma unroll
    for (int u = 0; u < kJoinRegs; ++u) {
        const int i = 4 * (threadIdx.x + u * kJoinThreads);
        if (i < hidden) {
            const float4 w = join_load4(a.w + i);
            x[u].x += v[u].x * inv * w.x;
            x[u].y += v[u].y * inv * w.y;
            x[u].z += v[u].z * inv * w.z;
            x[u].w += v[u].w * inv * w.w;
            join_store4(xr + i, x[u]);
            if (a.copy) join_store4((T*)a.copy + t * hidden + i, x[u]);
        }
    }
}

template <typename TY, typename T, bool EXPERTS>
__global__ void __launch_bounds__(kJoinThreads) join_norm_kernel(JoinArgs a) {
    extern __shared__ float row_sh[];
    __shared__ float scratch[33];
    lsb_pdl_launch_dependents();
    lsb_pdl_wait();
    const int hidden = a.hidden;
    const size_t t = blockIdx.x;
    float ss = 0.f;
    for (int i = threadIdx.x; i < hidden; i += kJoinThreads) {
        float v = a.bias ? a.bias[i] : 0.f;
        if (EXPERTS) {
            for (int k = 0; k < a.top; ++k) {
                const int p = a.pos[t * a.top + k];
                if (p >= 0 && p < a.capacity) v += a.wts[t * a.top + k] * lsb_to_float(((const TY*)a.y[0])[(size_t)p * hidden + i]);
            }
        } else {
            for (int b = 0; b < a.terms; ++b) v += a.s[b] * lsb_to_float(((const TY*)a.y[b])[t * hidden + i]);
        }
        row_sh[i] = v;
        ss += v * v;
    }
    const float inv = rsqrtf(lsb_block_sum(ss, scratch) / (float)hidden + a.eps);
    for (int i = threadIdx.x; i < hidden; i += kJoinThreads) {
        const float x = a.x[t * hidden + i] + row_sh[i] * inv * a.w[i];
        a.x[t * hidden + i] = x;
        if (a.copy) ((T*)a.copy)[t * hidden + i] = lsb_from_float<T>(x);
    }
}

LSB_API int lsb_join_max_terms() { return kMaxTerms; }

// x [rows, hidden] 32-bit, in place.  pos null: `terms` results ys[b] [rows, hidden] with factors; else the rows of
// ys[0] [capacity, hidden] that pos [rows, top] names, weighted by wts.  bias, copy may be null.
LSB_API int lsb_join_norm(float* x, const void* const* ys, const float* scales, int terms, int y_dtype, const float* bias,
                          const int* pos, const float* wts, int top, int capacity, const float* w, float eps, void* copy,
                          int copy_dtype, int rows, int hidden, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (terms < 1 || terms > kMaxTerms || hidden <= 0 || (pos && (terms != 1 || top <= 0 || !wts))) return (int)cudaErrorInvalidValue;
    JoinArgs a;
    a.x = x;
    a.terms = terms;
    bool vec = hidden % 4 == 0 && hidden <= 4 * kJoinRegs * kJoinThreads;
    for (int b = 0; b < kMaxTerms; ++b) {
        a.y[b] = b < terms ? ys[b] : nullptr;
        a.s[b] = b < terms ? scales[b] : 0.f;
        vec = vec && (uintptr_t)a.y[b] % 16 == 0;
    }
    for (const void* p : {(const void*)x, (const void*)bias, (const void*)w, (const void*)copy}) vec = vec && (uintptr_t)p % 16 == 0;
    a.bias = bias; a.pos = pos; a.wts = wts; a.top = top; a.capacity = capacity;
    a.w = w; a.eps = eps; a.copy = copy; a.hidden = hidden;
    const size_t smem = (size_t)hidden * sizeof(float);
    if (!vec && smem > 200 * 1024) return (int)cudaErrorInvalidValue;
#define LSB_JOIN(TY, E)                                                                                             \
    do {                                                                                                            \
        if (vec) return lsb_launch(join_norm_vec_kernel<TY, T, E>, dim3(rows), dim3(kJoinThreads), 0, stream, 1, a); \
        if (smem > 48 * 1024) {                                                                                     \
            int rc = (int)cudaFuncSetAttribute(join_norm_kernel<TY, T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
            if (rc) return rc;                                                                                      \
        }                                                                                                           \
        return lsb_launch(join_norm_kernel<TY, T, E>, dim3(rows), dim3(kJoinThreads), smem, stream, 1, a);          \
    } while (0)
    LSB_DISPATCH_DTYPE(copy_dtype, {
        if (y_dtype == LSB_F32) {
            if (pos) LSB_JOIN(float, true);
            else LSB_JOIN(float, false);
        } else {
            if (pos) LSB_JOIN(__nv_bfloat16, true);
            else LSB_JOIN(__nv_bfloat16, false);
        }
    });
#undef LSB_JOIN
    return 0;
}
