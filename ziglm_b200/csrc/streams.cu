// Residual streams (hyper-connections): a token is carried by s copies of the residual, x_1 .. x_s, float rows of
// s * d numbers.  Around a sublayer with learned numbers in [s], out [s] and mix [s, s] (indexed [from, to]):
//     u = sum_a in[a] x_a;   h = u / sqrt(mean u^2 + eps) * w;   y = sublayer(h);
//     x_b <- sum_a mix[a, b] x_a + out[b] y                         (every x on the right is an old one)
// stream_norm makes h.  stream_mix forms the new streams in place and, while their elements are in registers, the h of
// the sublayer that follows: one pass over the streams a sublayer.  y is one branch, or `factor` times the sum of two
// branches, each divided by its own root mean square over d and multiplied by a weight.
// One block a token.  All of it is float; only h has the step's type.
#include "common.cuh"

namespace zlm {

constexpr int ST_MAX = 16;           // streams

template <typename TO> __device__ __forceinline__ void st_store4(TO* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void st_store4<float>(float* p, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void st_store4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<uint32_t*>(&lo);
    v.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = v;
}

// W elements at a time: 4 where rows, widths and addresses allow it, else 1.
template <int W> struct StVec { float f[W]; };
template <int W> __device__ __forceinline__ StVec<W> st_load(const float* p) {
    StVec<W> v;
    if constexpr (W == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v.f[0] = t.x; v.f[1] = t.y; v.f[2] = t.z; v.f[3] = t.w;
    } else v.f[0] = *p;
    return v;
}
template <int W> __device__ __forceinline__ void st_put(float* p, const StVec<W>& v) {
    if constexpr (W == 4) *reinterpret_cast<float4*>(p) = make_float4(v.f[0], v.f[1], v.f[2], v.f[3]);
    else *p = v.f[0];
}
template <typename TO, int W> __device__ __forceinline__ void st_out(TO* p, const StVec<W>& v) {
    if constexpr (W == 4) st_store4<TO>(p, v.f[0], v.f[1], v.f[2], v.f[3]);
    else *p = from_float<TO>(v.f[0]);
}

// h rows from u (shared memory, d floats) and the sum of its squares over this thread's elements.
template <typename TO, int W>
__device__ __forceinline__ void st_norm_rows(const float* u_s, float ss, float* scratch, const float* __restrict__ w, float eps,
                                             TO* __restrict__ h, int d) {
    const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)d + eps);
    for (int i = threadIdx.x * W; i < d; i += blockDim.x * W) {
        const StVec<W> u = st_load<W>(u_s + i), ww = st_load<W>(w + i);
        StVec<W> r;
#pragma unroll
        for (int e = 0; e < W; ++e) r.f[e] = (u.f[e] * inv) * ww.f[e];
        st_out<TO, W>(h + i, r);
    }
}

// in null: every stream counts once (the sum of the streams).  rows null: row r of x; else row rows[r].
template <typename TO, int W>
__global__ void __launch_bounds__(256)
stream_norm_kernel(const float* __restrict__ x, const float* __restrict__ in, int s,
                                   const float* __restrict__ w, float eps, const int* __restrict__ rows, TO* __restrict__ h,
                                   int d) {
    extern __shared__ __align__(16) float st_sm[];
    __shared__ float scratch[33];
    pdl_launch_dependents();
    pdl_wait();
    const long r = rows != nullptr ? rows[blockIdx.x] : blockIdx.x;
    const float* xr = x + r * s * d;
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < d; i += blockDim.x * W) {
        StVec<W> u;
#pragma unroll
        for (int e = 0; e < W; ++e) u.f[e] = 0.f;
        for (int a = 0; a < s; ++a) {
            const StVec<W> v = st_load<W>(xr + (long)a * d + i);
            const float c = in != nullptr ? in[a] : 1.0f;
#pragma unroll
            for (int e = 0; e < W; ++e) u.f[e] = fmaf(c, v.f[e], u.f[e]);
        }
#pragma unroll
        for (int e = 0; e < W; ++e) ss = fmaf(u.f[e], u.f[e], ss);
        st_put<W>(st_sm + i, u);                           // read back by the thread that wrote it
    }
    st_norm_rows<TO, W>(st_sm, ss, scratch, w, eps, h + (long)blockIdx.x * d, d);
}

// coef: float [s * s + s], mix then out.  b2 null: y = b1.  h null: no rows for a following sublayer.
template <typename TO, int W, int S>
__global__ void __launch_bounds__(256)
stream_mix_kernel(float* __restrict__ x, const float* __restrict__ coef, int s_rt,
                                  const float* __restrict__ b1, const float* __restrict__ w1, const float* __restrict__ b2,
                                  const float* __restrict__ w2, float branch_eps, float factor,
                                  const float* __restrict__ next_in, const float* __restrict__ next_w, float next_eps,
                                  TO* __restrict__ h, int d) {
    extern __shared__ __align__(16) float st_sm[];
    __shared__ float scratch[33], coef_s[ST_MAX * ST_MAX + 2 * ST_MAX];
    constexpr int SA = S > 0 ? S : ST_MAX;
    const int s = S > 0 ? S : s_rt;
    pdl_launch_dependents();
    // the coefficients are weights: nothing of the step writes them
    for (int i = threadIdx.x; i < s * s + s; i += blockDim.x) coef_s[i] = coef[i];
    if (h != nullptr)
        for (int i = threadIdx.x; i < s; i += blockDim.x) coef_s[s * s + s + i] = next_in[i];
    pdl_wait();
    __syncthreads();
    const float* y1 = b1 + (long)blockIdx.x * d;
    const float* y2 = b2 != nullptr ? b2 + (long)blockIdx.x * d : nullptr;
    float* xr = x + (long)blockIdx.x * s * d;
    float f1 = 1.f, f2 = 0.f;
    if (y2 != nullptr) {
        float s1 = 0.f, s2 = 0.f;
        for (int i = threadIdx.x * W; i < d; i += blockDim.x * W) {
            const StVec<W> a = st_load<W>(y1 + i), b = st_load<W>(y2 + i);
#pragma unroll
            for (int e = 0; e < W; ++e) { s1 = fmaf(a.f[e], a.f[e], s1); s2 = fmaf(b.f[e], b.f[e], s2); }
        }
        f1 = factor / sqrtf(block_sum(s1, scratch) / (float)d + branch_eps);
        f2 = factor / sqrtf(block_sum(s2, scratch) / (float)d + branch_eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x * W; i < d; i += blockDim.x * W) {
        StVec<W> y = st_load<W>(y1 + i);
        if (y2 != nullptr) {
            const StVec<W> b = st_load<W>(y2 + i), v1 = st_load<W>(w1 + i), v2 = st_load<W>(w2 + i);
#pragma unroll
            for (int e = 0; e < W; ++e) y.f[e] = fmaf(y.f[e] * f1, v1.f[e], (b.f[e] * f2) * v2.f[e]);
        }
        StVec<W> old[SA], u;
#pragma unroll
        for (int a = 0; a < SA; ++a)
            if (a < s) old[a] = st_load<W>(xr + (long)a * d + i);
#pragma unroll
        for (int e = 0; e < W; ++e) u.f[e] = 0.f;
#pragma unroll
        for (int b = 0; b < SA; ++b) {
            if (b >= s) break;
            StVec<W> v;
            const float co = coef_s[s * s + b];
#pragma unroll
            for (int e = 0; e < W; ++e) v.f[e] = co * y.f[e];
#pragma unroll
            for (int a = 0; a < SA; ++a) {
                if (a >= s) break;
                const float cm = coef_s[a * s + b];
#pragma unroll
                for (int e = 0; e < W; ++e) v.f[e] = fmaf(cm, old[a].f[e], v.f[e]);
            }
            st_put<W>(xr + (long)b * d + i, v);
            if (h != nullptr) {
                const float ci = coef_s[s * s + s + b];
#pragma unroll
                for (int e = 0; e < W; ++e) u.f[e] = fmaf(ci, v.f[e], u.f[e]);
            }
        }
        if (h != nullptr) {
#pragma unroll
            for (int e = 0; e < W; ++e) ss = fmaf(u.f[e], u.f[e], ss);
            st_put<W>(st_sm + i, u);
        }
    }
    if (h != nullptr) st_norm_rows<TO, W>(st_sm, ss, scratch, next_w, next_eps, h + (long)blockIdx.x * d, d);
}

// Every stream of a token starts as its row of the table.
template <typename TW>
__global__ void embed_streams_kernel(const TW* __restrict__ table, const int* __restrict__ tokens, float* __restrict__ out,
                                     int s, int d, float scale) {
    pdl_launch_dependents();
    pdl_wait();
    const TW* row = table + (long)tokens[blockIdx.x] * d;
    float* o = out + (long)blockIdx.x * s * d;
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        const float v = to_float(row[i]) * scale;
        for (int a = 0; a < s; ++a) o[(long)a * d + i] = v;
    }
}

static inline int st_threads(int d, int w) {
    const int units = (d + w - 1) / w;
    return units >= 512 ? 256 : (units >= 256 ? 128 : 64);
}
static inline bool st_aligned(const void* p) { return (uintptr_t)p % 16 == 0; }

}  // namespace zlm

using namespace zlm;

// x: float [rows][s * d]; in: float [s] or null; w: float [d]; h: [n_rows][d] in h_dtype.
ZLM_EXPORT int zlm_stream_norm(const float* x, const float* in, int s, const float* w, float eps, const int* rows, void* h,
                               int h_dtype, int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (d <= 0 || s <= 0 || s > ST_MAX) return ZLM_ERR_BAD_ARG;
    const size_t smem = (size_t)d * sizeof(float);
    if (smem > 48 * 1024 - 1024) return ZLM_ERR_UNSUPPORTED;
    const bool vec = d % 4 == 0 && st_aligned(x) && st_aligned(w) && st_aligned(h);
    const int threads = st_threads(d, vec ? 4 : 1);
    cudaError_t e;
#define ZLM_SN(TO, W)                                                                                                  \
    e = launch_pdl(stream_norm_kernel<TO, W>, dim3(n_rows), dim3(threads), smem, stream, x, in, s, w, eps, rows, (TO*)h, d)
    if (h_dtype == ZLM_F32) { if (vec) ZLM_SN(float, 4); else ZLM_SN(float, 1); }
    else if (h_dtype == ZLM_BF16) { if (vec) ZLM_SN(__nv_bfloat16, 4); else ZLM_SN(__nv_bfloat16, 1); }
    else return ZLM_ERR_UNSUPPORTED;
#undef ZLM_SN
    return e == cudaSuccess ? launch_status() : (int)e;
}

// x: float [n_rows][s * d], in place; coef: float [s * s + s] (mix [from][to], then out); b1, b2: float [n_rows][d] (b2, w1,
// w2 null: y = b1); next_in float [s], next_w float [d] and h [n_rows][d] of the sublayer that follows, or null.
ZLM_EXPORT int zlm_stream_mix(float* x, const float* coef, int s, const float* b1, const float* w1, const float* b2,
                              const float* w2, float branch_eps, float factor, const float* next_in, const float* next_w,
                              float next_eps, void* h, int h_dtype, int n_rows, int d, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (d <= 0 || s <= 0 || s > ST_MAX || (b2 != nullptr && (w1 == nullptr || w2 == nullptr)) ||
        (h != nullptr && (next_in == nullptr || next_w == nullptr)))
        return ZLM_ERR_BAD_ARG;
    const size_t smem = h != nullptr ? (size_t)d * sizeof(float) : 0;
    if (smem > 48 * 1024 - 2048) return ZLM_ERR_UNSUPPORTED;
    const bool vec = d % 4 == 0 && st_aligned(x) && st_aligned(b1) && st_aligned(w1) && st_aligned(b2) && st_aligned(w2) &&
                     st_aligned(next_w) && st_aligned(h);
    const int threads = st_threads(d, vec ? 4 : 1);
    cudaError_t e;
#define ZLM_SM(TO, W, S)                                                                                               \
    e = launch_pdl(stream_mix_kernel<TO, W, S>, dim3(n_rows), dim3(threads), smem, stream, x, coef, s, b1, w1, b2, w2,   \
                   branch_eps, factor, next_in, next_w, next_eps, (TO*)h, d)
#define ZLM_SM_S(TO, W)                                                                                                \
    switch (s) {                                                                                                       \
        case 1: ZLM_SM(TO, W, 1); break;                                                                               \
        case 2: ZLM_SM(TO, W, 2); break;                                                                               \
        case 3: ZLM_SM(TO, W, 3); break;                                                                               \
        case 4: ZLM_SM(TO, W, 4); break;                                                                               \
        default: ZLM_SM(TO, W, 0); break;                                                                              \
    }
    if (h == nullptr || h_dtype == ZLM_F32) { if (vec) { ZLM_SM_S(float, 4) } else { ZLM_SM_S(float, 1) } }
    else if (h_dtype == ZLM_BF16) { if (vec) { ZLM_SM_S(__nv_bfloat16, 4) } else { ZLM_SM_S(__nv_bfloat16, 1) } }
    else return ZLM_ERR_UNSUPPORTED;
#undef ZLM_SM_S
#undef ZLM_SM
    return e == cudaSuccess ? launch_status() : (int)e;
}

// out: float [T][s * d]: s copies of float(table[tokens[t]]) * scale.
ZLM_EXPORT int zlm_embed_streams(const void* table, int table_dtype, const int* tokens, float* out, int T, int s, int d,
                                 float scale, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || s <= 0) return ZLM_ERR_BAD_ARG;
    const int threads = d >= 1024 ? 256 : 128;
    cudaError_t e;
    if (table_dtype == ZLM_F32)
        e = launch_pdl(embed_streams_kernel<float>, dim3(T), dim3(threads), 0, stream, (const float*)table, tokens, out, s, d, scale);
    else if (table_dtype == ZLM_BF16)
        e = launch_pdl(embed_streams_kernel<__nv_bfloat16>, dim3(T), dim3(threads), 0, stream, (const __nv_bfloat16*)table, tokens,
                       out, s, d, scale);
    else
        return ZLM_ERR_UNSUPPORTED;
    return e == cudaSuccess ? launch_status() : (int)e;
}
