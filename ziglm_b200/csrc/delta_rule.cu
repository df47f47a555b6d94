// The gated delta rule over a step's sequences, with the state carried in float.  Per head, with unit vectors q, k of D
// elements (q also times D^-1/2), values v of V elements, a write strength beta and decays g (one a head, or one a key
// channel) the state S [D, V] moves as
//     S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// q, k and v are columns of a projection's rows behind a short causal convolution a channel and silu; heads share the
// q and k of their group (H heads over G groups).  g = exp(-rate_h softplus(a + dt_bias)), beta = sigmoid(b).
//
// What a sequence carries: the last inputs of the convolution, and S.
//   ring  float [slots][K][C]       row p mod K holds the inputs of position p (C channels: q, k, v as they lie in the
//                                   projection).  A ring of K rows: the row a step of one token writes is one no block of
//                                   that step reads, so blocks that share the channels of q and k need no order.
//   S     float [slots][H][V][Dp]   transposed, so that a value column's D elements are contiguous; Dp: D rounded up to a
//                                   multiple of 4, the elements behind D stay zero.
//
// A step of one token a sequence is one kernel (dr_decode): a block takes a (sequence, head), asks for its part of S
// before it waits for the projection, makes q, k, v, g and beta, updates S in place, norms the head's output over V,
// applies weight and gate and writes the rows the output projection reads.
//
// Any other step is three kernels, over chunks of DR_C tokens of a sequence.  dr_prep makes q, k, v, g, beta of every
// token in float and writes the ring.  Behind a state S0 a chunk unrolls to (products of decays: from where to where)
//     R_t = (G_0t k_t) . S0            A_tj = beta_t (G_jt k_t) . k_j   (j < t)     u = (I + A)^-1 beta (v - R)
//     o_t = (G_0t q_t) . S0 + sum_(j <= t) B_tj u_j,  B_tj = (G_jt q_t) . k_j       S = G_0n S0 + sum_j (G_jn k_j) u_j^T
// with G_jt the product of the decays of the tokens behind j up to t: never a quotient, so a strong decay is a zero and not
// an overflow.  dr_chunk makes everything of this that does not depend on S, all chunks and heads side by side: the
// weighted keys and queries, T = (I + A)^-1 diag(beta) and B.  dr_scan walks the chunks with S in registers, so a chunk is
// three float products of which none waits for the token before: a column of S is spread over 16 lanes of a warp, a
// lane holding two or four columns, the columns of a head over blocks, which need nothing from each other; the sums over the
// lanes are scattered so that lane (t, column) ends with R_t and o_t of its column.  The chunks come through shared memory
// (cp.async, three stages).  Every sum is float FMA (two at a time, fma.rn.f32x2); nothing that enters the recurrence
// passes through a 16-bit type behind the projection.
#include "common.cuh"

namespace zlm {

constexpr int DR_C = 8;              // tokens of a chunk
constexpr int DR_L = 16;             // lanes that share a column of the state in dr_scan
constexpr int DR_THREADS = 128;      // of dr_chunk: DR_C tokens x DR_L lanes
constexpr int DR_VT = 16;            // value columns of a block of dr_scan
constexpr int DR_PREP_WARPS = 4;
constexpr int DR_SLIDE = 4;          // taps dr_prep keeps in registers

__device__ __forceinline__ float dr_softplus(float z) { return z > 20.f ? z : log1pf(expf(z)); }
__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float dr_silu(float z) { return z / (1.0f + expf(-z)); }

template <typename T> __device__ __forceinline__ float4 dr_load4(const T* p);
template <> __device__ __forceinline__ float4 dr_load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 dr_load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

// What the kernels read of the projection and of the sequence's state.
template <typename T>
struct DrIn {
    const T* proj;              // [T rows] with stride proj_stride; q | k | v start at column 0: C = 2 G D + H V channels
    long proj_stride;
    const float* taps;          // [K][C], the current token's row last
    float* ring;                // [slots][K][C]
    int H, G, D, V, C, K, Dp, Vp;
    const float* a;             // rows with stride a_stride: H numbers, or H * D with a decay a channel
    long a_stride;
    const float* b;             // rows with stride b_stride: H numbers
    long b_stride;
    const float* rate;          // [H]: exp(A_log)
    const float* dt_bias;       // [H] or [H * D]
    const int* slots;
    const int* past_lens;
    const int* cu_seqlens;
};

// The convolution of one channel for the token at index i of its sequence's tokens of this step (position pos).
template <typename T>
__device__ __forceinline__ float dr_conv1(const DrIn<T>& in, const T* __restrict__ x, const float* __restrict__ ring, int i,
                                          int pos, int c) {
    float acc = 0.f;
    for (int j = in.K - 1; j >= 0; --j) {                // oldest input first
        float xv = 0.f;
        if (i - j >= 0) xv = to_float(x[-(long)j * in.proj_stride + c]);
        else if (pos - j >= 0) xv = ring[(long)((pos - j) % in.K) * in.C + c];
        acc = fmaf(in.taps[(long)(in.K - 1 - j) * in.C + c], xv, acc);
    }
    return acc;
}
template <typename T>
__device__ __forceinline__ float4 dr_conv4(const DrIn<T>& in, const T* __restrict__ x, const float* __restrict__ ring, int i,
                                           int pos, int c) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = in.K - 1; j >= 0; --j) {
        float4 xv = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i - j >= 0) xv = dr_load4<T>(x - (long)j * in.proj_stride + c);
        else if (pos - j >= 0) xv = *reinterpret_cast<const float4*>(ring + (long)((pos - j) % in.K) * in.C + c);
        const float4 w = *reinterpret_cast<const float4*>(in.taps + (long)(in.K - 1 - j) * in.C + c);
        acc.x = fmaf(w.x, xv.x, acc.x); acc.y = fmaf(w.y, xv.y, acc.y);
        acc.z = fmaf(w.z, xv.z, acc.z); acc.w = fmaf(w.w, xv.w, acc.w);
    }
    return acc;
}

// ------------------------------------------------------------------------------------------------ prompt steps
// grid (tiles of `tile` tokens, units / warps, sequences).  A warp takes one unit for the tile's tokens: a q head, a k
// head, a v head, or the decays and the write strength of a head.  The first tile of a sequence, which alone reads the
// ring (tile >= K - 1), writes it when it has: the last inputs of the step come from the projection.
template <typename T, bool VEC>
__global__ void __launch_bounds__(DR_PREP_WARPS * 32)
dr_prep_kernel(DrIn<T> in, int channel_decay, int tile, float* __restrict__ qk_out, float* __restrict__ v_out,
               float* __restrict__ g_out, float* __restrict__ beta_out) {
    extern __shared__ float dr_sm[];
    pdl_wait();
    const int b = blockIdx.z;
    const int first = in.cu_seqlens[b], n_new = in.cu_seqlens[b + 1] - first;
    const int lo = blockIdx.x * tile, hi = min(n_new, lo + tile);
    if (lo >= n_new) return;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int unit = blockIdx.y * DR_PREP_WARPS + warp;
    const int n_conv = 2 * in.G + in.H;
    if (unit >= n_conv + in.H) return;
    if (unit >= n_conv) {
        const int h = unit - n_conv;
        const float rate = in.rate[h];
        for (int i = lo; i < hi; ++i) {
            const long t = first + i;
            if (lane == 0) beta_out[t * in.H + h] = dr_sigmoid(in.b[t * in.b_stride + h]);
            if (channel_decay && VEC && in.a_stride % 4 == 0 && (uintptr_t)in.a % 16 == 0) {
                for (int c = lane * 4; c < in.D; c += 128) {
                    const float4 a4 = *reinterpret_cast<const float4*>(in.a + t * in.a_stride + (long)h * in.D + c);
                    const float4 d4 = *reinterpret_cast<const float4*>(in.dt_bias + h * in.D + c);
                    *reinterpret_cast<float4*>(g_out + (t * in.H + h) * in.Dp + c) =
                        make_float4(expf(-rate * dr_softplus(a4.x + d4.x)), expf(-rate * dr_softplus(a4.y + d4.y)),
                                    expf(-rate * dr_softplus(a4.z + d4.z)), expf(-rate * dr_softplus(a4.w + d4.w)));
                }
            } else if (channel_decay) {
                for (int c = lane; c < in.Dp; c += 32)
                    g_out[(t * in.H + h) * in.Dp + c] = c < in.D
                        ? expf(-rate * dr_softplus(in.a[t * in.a_stride + (long)h * in.D + c] + in.dt_bias[h * in.D + c])) : 0.f;
            } else if (lane == 0) {
                g_out[t * in.H + h] = expf(-rate * dr_softplus(in.a[t * in.a_stride + h] + in.dt_bias[h]));
            }
        }
        return;
    }
    const bool is_v = unit >= 2 * in.G;
    const int size = is_v ? in.V : in.D, padded = is_v ? in.Vp : in.Dp;
    const int c0 = is_v ? 2 * in.G * in.D + (unit - 2 * in.G) * in.V : unit * in.D;
    float* ring = in.ring + (long)in.slots[b] * in.K * in.C;
    const int past = in.past_lens[b];
    float* row_s = dr_sm + warp * in.Dp;                  // a q or k head before its norm
    const float q_scale = unit < in.G ? 1.0f / sqrtf((float)in.D) : 1.0f;
    const bool slid = VEC && in.K <= DR_SLIDE && size <= 128;
    if constexpr (VEC) {
        // a lane's four channels, the inputs of the last tokens in registers
        if (slid) {
            const int c = lane * 4;
            const bool on = c < size;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            float4 w[DR_SLIDE], win[DR_SLIDE];                // of the token j places back: its tap and its input
#pragma unroll
            for (int j = 0; j < DR_SLIDE; ++j) {
                w[j] = on && j < in.K ? *reinterpret_cast<const float4*>(in.taps + (long)(in.K - 1 - j) * in.C + c0 + c) : zero;
                win[j] = zero;
            }
            auto input = [&](int i) {                         // of the token at index i of the step, or of one before the step
                if (!on || past + i < 0) return zero;
                return i >= 0 ? dr_load4<T>(in.proj + (long)(first + i) * in.proj_stride + c0 + c)
                              : *reinterpret_cast<const float4*>(ring + (long)((past + i) % in.K) * in.C + c0 + c);
            };
#pragma unroll
            for (int j = DR_SLIDE - 1; j > 0; --j)
                if (j < in.K) win[j - 1] = input(lo - j);
#pragma unroll 4
            for (int i = lo; i < hi; ++i) {
                const long t = first + i;
#pragma unroll
                for (int j = DR_SLIDE - 1; j > 0; --j) win[j] = win[j - 1];
                win[0] = input(i);
                float4 y = zero;
#pragma unroll
                for (int j = DR_SLIDE - 1; j >= 0; --j) {
                    y.x = fmaf(w[j].x, win[j].x, y.x); y.y = fmaf(w[j].y, win[j].y, y.y);
                    y.z = fmaf(w[j].z, win[j].z, y.z); y.w = fmaf(w[j].w, win[j].w, y.w);
                }
                y.x = dr_silu(y.x); y.y = dr_silu(y.y); y.z = dr_silu(y.z); y.w = dr_silu(y.w);
                if (is_v) {
                    if (on) *reinterpret_cast<float4*>(v_out + (t * in.H + (unit - 2 * in.G)) * in.Vp + c) = y;
                    continue;
                }
                const float ss = fmaf(y.x, y.x, fmaf(y.y, y.y, fmaf(y.z, y.z, y.w * y.w)));
                const float inv = q_scale / sqrtf(warp_sum(ss) + 1e-6f);
                if (on)
                    *reinterpret_cast<float4*>(qk_out + (t * 2 * in.G + unit) * in.Dp + c) =
                        make_float4(y.x * inv, y.y * inv, y.z * inv, y.w * inv);
            }
        }
    }
    for (int i = slid ? hi : lo; i < hi; ++i) {
        const long t = first + i;
        const T* x = in.proj + t * in.proj_stride;
        float* dst = is_v ? v_out + (t * in.H + (unit - 2 * in.G)) * in.Vp : qk_out + (t * 2 * in.G + unit) * in.Dp;
        float ss = 0.f;
        if constexpr (VEC) {
            for (int c = lane * 4; c < size; c += 128) {
                float4 y = dr_conv4<T>(in, x, ring, i, past + i, c0 + c);
                y.x = dr_silu(y.x); y.y = dr_silu(y.y); y.z = dr_silu(y.z); y.w = dr_silu(y.w);
                if (is_v) *reinterpret_cast<float4*>(dst + c) = y;
                else {
                    ss = fmaf(y.x, y.x, ss); ss = fmaf(y.y, y.y, ss); ss = fmaf(y.z, y.z, ss); ss = fmaf(y.w, y.w, ss);
                    *reinterpret_cast<float4*>(row_s + c) = y;
                }
            }
        } else {
            for (int c = lane; c < padded; c += 32) {
                const float y = c < size ? dr_silu(dr_conv1<T>(in, x, ring, i, past + i, c0 + c)) : 0.f;
                if (is_v) dst[c] = y;
                else { ss = fmaf(y, y, ss); row_s[c] = y; }
            }
        }
        if (is_v) continue;
        const float inv = q_scale / sqrtf(warp_sum(ss) + 1e-6f);
        if constexpr (VEC) {
            for (int c = lane * 4; c < size; c += 128) {
                float4 y = *reinterpret_cast<const float4*>(row_s + c);
                y.x *= inv; y.y *= inv; y.z *= inv; y.w *= inv;
                *reinterpret_cast<float4*>(dst + c) = y;
            }
        } else {
            for (int c = lane; c < padded; c += 32) dst[c] = row_s[c] * inv;
        }
    }
    if (lo != 0) return;
    // the ring: the step's last K inputs, each in its position's row (a lane writes the channels it has read)
    const T* last_row = in.proj + (long)(first + n_new - 1) * in.proj_stride;
    for (int j = min(in.K, n_new) - 1; j >= 0; --j) {
        float* row = ring + (long)((past + n_new - 1 - j) % in.K) * in.C + c0;
        const T* x = last_row - (long)j * in.proj_stride + c0;
        if constexpr (VEC) {
            for (int c = lane * 4; c < size; c += 128) *reinterpret_cast<float4*>(row + c) = dr_load4<T>(x + c);
        } else {
            for (int c = lane; c < size; c += 32) row[c] = to_float(x[c]);
        }
    }
}

__device__ __forceinline__ void dr_cp16(float* smem, const float* gmem) {
    const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem) : "memory");
}
__device__ __forceinline__ void dr_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void dr_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <int L> __device__ __forceinline__ float dr_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// The place of a chunk among all chunks of the step: sequence b's chunks lie behind those of the sequences before it.
__device__ __forceinline__ long dr_chunk_index(int first, int b, int chunk) { return (long)(first / DR_C) + b + chunk; }

// What dr_chunk leaves of a (chunk, head), in floats, rows padded with zeros to DS elements:
//   G_0t k_t [DR_C][DS], G_0t q_t [DR_C][DS], G_jn k_j [DR_C][DS], G_0n [DS], then per token its row of T and of B [DR_C][2 DR_C]
// Tokens behind the end of a short chunk are zero in all of them.
__host__ __device__ constexpr int dr_record(int NI) { return (3 * DR_C + 1) * 64 * NI + 2 * DR_C * DR_C; }

// grid (chunks of the longest sequence, heads, sequences); thread (j, l): token j of the chunk, lane l of its D elements.
// qk: float [T][2 G][Dp]; g: [T][H][Dp] (CH) or [T][H]; beta: [T][H]; rec: [chunks][H] records.
template <int NI, bool CH>
__global__ void __launch_bounds__(DR_THREADS)
dr_chunk_kernel(const float* __restrict__ qk, const float* __restrict__ g, const float* __restrict__ beta,
                const int* __restrict__ cu_seqlens, float* __restrict__ rec, int H, int G, int Dp) {
    constexpr int D4 = DR_L * NI;                          // float4 of a padded row
    extern __shared__ __align__(16) float dr_sm[];
    float4* k4 = reinterpret_cast<float4*>(dr_sm);         // [DR_C][D4]
    float4* q4 = k4 + DR_C * D4;
    float4* g4 = q4 + DR_C * D4;                           // CH
    __shared__ float a_s[DR_C][DR_C], b_s[DR_C][DR_C], g_s[DR_C], beta_s[DR_C];
    pdl_wait();
    const int b = blockIdx.z, h = blockIdx.y, kv = h / (H / G);
    const int first = cu_seqlens[b], n_new = cu_seqlens[b + 1] - first;
    const int at = blockIdx.x * DR_C, n = min(DR_C, n_new - at);
    if (n <= 0) return;
    const int tid = threadIdx.x, j = tid / DR_L, l = tid % DR_L, d4 = Dp / 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const long t0 = first + at;
    // a token's row by the lanes that work on it
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int c = l + DR_L * i;
        const bool in = j < n && c < d4;
        k4[j * D4 + c] = in ? reinterpret_cast<const float4*>(qk + ((t0 + j) * 2 * G + G + kv) * Dp)[c] : zero;
        q4[j * D4 + c] = in ? reinterpret_cast<const float4*>(qk + ((t0 + j) * 2 * G + kv) * Dp)[c] : zero;
        if constexpr (CH) g4[j * D4 + c] = in ? reinterpret_cast<const float4*>(g + ((t0 + j) * H + h) * Dp)[c] : zero;
    }
    if (tid < DR_C) {
        beta_s[tid] = tid < n ? beta[(t0 + tid) * H + h] : 0.f;
        if constexpr (!CH) g_s[tid] = tid < n ? g[(t0 + tid) * H + h] : 0.f;
    }
    if (tid < DR_C * DR_C) (&a_s[0][0])[tid] = (&b_s[0][0])[tid] = 0.f;
    __syncthreads();
    // token j's key, decayed from one later token to the next: its products with their k and q
    float4 w[NI];
    float wsc = 1.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) w[i] = k4[j * D4 + l + DR_L * i];
    for (int t = 0; t < n; ++t) {                          // every thread takes every round: shuffles inside
        float ka = 0.f, qa = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 kk = k4[t * D4 + l + DR_L * i], qq = q4[t * D4 + l + DR_L * i];
            if constexpr (CH) {
                if (t > j) {
                    const float4 gg = g4[t * D4 + l + DR_L * i];
                    w[i].x *= gg.x; w[i].y *= gg.y; w[i].z *= gg.z; w[i].w *= gg.w;
                }
            }
            ka = fmaf(kk.x, w[i].x, ka); ka = fmaf(kk.y, w[i].y, ka); ka = fmaf(kk.z, w[i].z, ka); ka = fmaf(kk.w, w[i].w, ka);
            qa = fmaf(qq.x, w[i].x, qa); qa = fmaf(qq.y, w[i].y, qa); qa = fmaf(qq.z, w[i].z, qa); qa = fmaf(qq.w, w[i].w, qa);
        }
        if constexpr (!CH) { if (t > j) wsc *= g_s[t]; }
        ka = dr_sum<DR_L>(ka);
        qa = dr_sum<DR_L>(qa);
        if (t >= j && l == 0) {
            b_s[t][j] = qa * wsc;
            if (t > j) a_s[t][j] = beta_s[t] * (ka * wsc);
        }
    }
    float4* r4 = reinterpret_cast<float4*>(rec + (dr_chunk_index(first, b, blockIdx.x) * H + h) * dr_record(NI));
    {
        // decays from the state to token j, and from token j to the chunk's end (what w has become); a row behind a short
        // chunk's last token is zero because its k and q are
        float4 G0[NI];
        float g0 = 1.f;
        if constexpr (CH) {
#pragma unroll
            for (int i = 0; i < NI; ++i) G0[i] = g4[l + DR_L * i];
            for (int t = 1; t <= j; ++t) {
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const float4 gg = g4[t * D4 + l + DR_L * i];
                    G0[i].x *= gg.x; G0[i].y *= gg.y; G0[i].z *= gg.z; G0[i].w *= gg.w;
                }
            }
        } else {
            for (int t = 0; t <= j; ++t) g0 *= g_s[t];
        }
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int c = j * D4 + l + DR_L * i;
            const float4 gg = CH ? G0[i] : make_float4(g0, g0, g0, g0);
            const float4 kk = k4[c], qq = q4[c];
            r4[c] = make_float4(gg.x * kk.x, gg.y * kk.y, gg.z * kk.z, gg.w * kk.w);
            r4[DR_C * D4 + c] = make_float4(gg.x * qq.x, gg.y * qq.y, gg.z * qq.z, gg.w * qq.w);
            r4[2 * DR_C * D4 + c] = make_float4(w[i].x * wsc, w[i].y * wsc, w[i].z * wsc, w[i].w * wsc);
            if (j == n - 1) r4[3 * DR_C * D4 + l + DR_L * i] = gg;
        }
    }
    __syncthreads();
    // column c of T: (I + A) x = beta_c e_c, downwards
    float* tb = reinterpret_cast<float*>(r4 + (3 * DR_C + 1) * D4);
    if (tid < DR_C) {
        float x[DR_C];
#pragma unroll
        for (int t = 0; t < DR_C; ++t) {
            float acc = t == tid ? beta_s[t] : 0.f;
#pragma unroll
            for (int u = 0; u < t; ++u) acc = fmaf(-a_s[t][u], x[u], acc);
            x[t] = acc;
            tb[t * 2 * DR_C + tid] = acc;                  // behind the last token: beta and A are zero, so is T
        }
    } else if (tid >= 64) {
        const int i = tid - 64, t = i / DR_C;
        tb[t * 2 * DR_C + DR_C + i % DR_C] = b_s[t][i % DR_C];
    }
}

// Two floats at a time.
typedef unsigned long long dr_f2;
__device__ __forceinline__ dr_f2 dr_fma2(dr_f2 a, dr_f2 b, dr_f2 c) {
    dr_f2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ dr_f2 dr_mul2(dr_f2 a, dr_f2 b) {
    dr_f2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ dr_f2 dr_pack2(float x, float y) {
    dr_f2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
    return d;
}
__device__ __forceinline__ float dr_both(dr_f2 v) {
    float x, y;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(v));
    return x + y;
}

// The sums over 16 lanes of N numbers a lane, scattered: lane l is left with those of numbers l N/16 .. in front.  Two sets
// side by side, so that the rounds of one hide those of the other.
template <int N>
__device__ __forceinline__ void dr_scatter(float (&a)[N], float (&b)[N], int l) {
#pragma unroll
    for (int o = 8, half = N / 2; o > 0; o >>= 1, half >>= 1) {
        const bool up = (l & o) != 0;
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float give = up ? a[i] : a[i + half], keep = up ? a[i + half] : a[i];
            a[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
#pragma unroll
        for (int i = 0; i < half; ++i) {
            const float give = up ? b[i] : b[i + half], keep = up ? b[i + half] : b[i];
            b[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
}

constexpr int DR_STAGES = 3;
// floats of a stage: the chunk's record and its values
__host__ __device__ constexpr int dr_stage(int NI) { return dr_record(NI) + DR_C * DR_VT; }

// A lane holds VC columns: what a lane reads of a chunk's rows from shared memory, which sets the pace, serves all of them.
// The threads of a block: two times VC columns a warp, DR_VT columns in all.
__host__ __device__ constexpr int dr_scan_threads(int VC) { return 32 * DR_VT / (2 * VC); }

// grid (value tiles, heads, sequences).  rec: the records of dr_chunk; v: [T][H][Vp]; out: float rows of H V numbers.
template <int NI, int VC>
__global__ void __launch_bounds__(dr_scan_threads(VC))
dr_scan_kernel(const float* __restrict__ rec, const float* __restrict__ v, float* __restrict__ state,
               const int* __restrict__ slots, const int* __restrict__ cu_seqlens, float* __restrict__ out, long out_stride, int H,
               int Dp, int V, int Vp) {
    constexpr int D4 = 16 * NI, STAGE = dr_stage(NI), RECORD = dr_record(NI), THREADS = dr_scan_threads(VC), X = VC / 2;
    extern __shared__ __align__(16) float dr_sm[];
    const int tid = threadIdx.x, lane = tid & 31, l = lane & 15;
    const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * DR_VT;
    const int d4 = Dp / 4;
    const int col0 = ((tid >> 5) * 2 + (lane >> 4)) * VC;   // this lane's columns of the tile
    const int my_t = l >> 1, my_col = col0 + (l & 1) * X;   // what the scattered sums leave this lane with: X columns of a token
    // values that are never fetched (behind a short chunk's last token, behind the last column) meet zeros: finite they must be
    for (int i = tid; i < DR_STAGES * DR_C * DR_VT; i += THREADS)
        dr_sm[(i / (DR_C * DR_VT)) * STAGE + RECORD + i % (DR_C * DR_VT)] = 0.f;
    float* st = state + ((long)slots[b] * H + h) * V * Dp;
    dr_f2 S[VC][2 * NI];
#pragma unroll
    for (int c = 0; c < VC; ++c) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            ulonglong2 s = make_ulonglong2(0, 0);
            if (v0 + col0 + c < V && l + DR_L * i < d4)
                s = reinterpret_cast<const ulonglong2*>(st + (long)(v0 + col0 + c) * Dp)[l + DR_L * i];
            S[c][2 * i] = s.x; S[c][2 * i + 1] = s.y;
        }
    }
    pdl_wait();
    __syncthreads();
    const int first = cu_seqlens[b], n_new = cu_seqlens[b + 1] - first;
    const int n_chunks = (n_new + DR_C - 1) / DR_C;
    const float* recs = rec + (dr_chunk_index(first, b, 0) * H + h) * RECORD;
    const int vj = tid / (DR_VT / 4), vi = 4 * (tid % (DR_VT / 4));            // what a thread fetches of the values
    const float* vsrc = v + ((first + vj) * (long)H + h) * Vp + v0 + vi;
    auto fetch = [&](int chunk) {
        if (chunk < n_chunks) {
            float* sm = dr_sm + (chunk % DR_STAGES) * STAGE;
            const float* src = recs + (long)chunk * H * RECORD;
#pragma unroll
            for (int i = 0; i < RECORD / 4; i += THREADS)
                if (i + tid < RECORD / 4) dr_cp16(sm + 4 * (i + tid), src + 4 * (i + tid));
            if (vj < min(DR_C, n_new - chunk * DR_C) && v0 + vi < Vp)
                dr_cp16(sm + RECORD + vj * DR_VT + vi, vsrc + (long)chunk * DR_C * H * Vp);
        }
        dr_cp_commit();
    };
    fetch(0);
    fetch(1);
    for (int chunk = 0; chunk < n_chunks; ++chunk) {
        dr_cp_wait<1>();
        __syncthreads();                                   // this chunk is here, and everyone is done with the one before
        fetch(chunk + 2);
        const float* sm = dr_sm + (chunk % DR_STAGES) * STAGE;
        const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(sm) + l;
        const ulonglong2* q2 = k2 + DR_C * D4;
        const ulonglong2* e2 = q2 + DR_C * D4;
        const ulonglong2* g2 = e2 + DR_C * D4;
        const float* tb_s = sm + (3 * DR_C + 1) * 4 * D4 + my_t * 2 * DR_C;      // this lane's row of T, then of B
        float R[DR_C * VC], O[DR_C * VC];
        // the chunk's keys and queries on the state
#pragma unroll
        for (int t = 0; t < DR_C; ++t) {
            dr_f2 r[VC], o[VC];
#pragma unroll
            for (int c = 0; c < VC; ++c) r[c] = o[c] = 0;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const ulonglong2 kk = k2[t * D4 + DR_L * i], qq = q2[t * D4 + DR_L * i];
#pragma unroll
                for (int c = 0; c < VC; ++c) {
                    r[c] = dr_fma2(kk.x, S[c][2 * i], r[c]); o[c] = dr_fma2(qq.x, S[c][2 * i], o[c]);
                    r[c] = dr_fma2(kk.y, S[c][2 * i + 1], r[c]); o[c] = dr_fma2(qq.y, S[c][2 * i + 1], o[c]);
                }
            }
#pragma unroll
            for (int c = 0; c < VC; ++c) { R[VC * t + c] = dr_both(r[c]); O[VC * t + c] = dr_both(o[c]); }
        }
        // the state before the chunk's writes
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const ulonglong2 gg = g2[DR_L * i];
#pragma unroll
            for (int c = 0; c < VC; ++c) {
                S[c][2 * i] = dr_mul2(S[c][2 * i], gg.x);
                S[c][2 * i + 1] = dr_mul2(S[c][2 * i + 1], gg.y);
            }
        }
        dr_scatter<DR_C * VC>(R, O, l);
        float e[X], u[X];
#pragma unroll
        for (int x = 0; x < X; ++x) {
            e[x] = sm[RECORD + my_t * DR_VT + my_col + x] - R[x];
            u[x] = 0.f;
        }
        // u = T e: a lane takes row t for its columns
        {
            const float4 t0 = *reinterpret_cast<const float4*>(tb_s), t1 = *reinterpret_cast<const float4*>(tb_s + 4);
            const float tr[DR_C] = {t0.x, t0.y, t0.z, t0.w, t1.x, t1.y, t1.z, t1.w};
            const int base = (lane & 16) | (l & 1);
#pragma unroll
            for (int j = 0; j < DR_C; ++j) {
#pragma unroll
                for (int x = 0; x < X; ++x) u[x] = fmaf(tr[j], __shfl_sync(0xffffffffu, e[x], base + 2 * j), u[x]);
            }
        }
        // o += B u, and the state: G_0n S + sum_j (G_jn k_j) u_j
        {
            const float4 t0 = *reinterpret_cast<const float4*>(tb_s + DR_C), t1 = *reinterpret_cast<const float4*>(tb_s + DR_C + 4);
            const float br[DR_C] = {t0.x, t0.y, t0.z, t0.w, t1.x, t1.y, t1.z, t1.w};
            const int base = lane & 16;
#pragma unroll
            for (int j = 0; j < DR_C; ++j) {
                float uc[VC];
                dr_f2 p[VC];
#pragma unroll
                for (int c = 0; c < VC; ++c) {
                    uc[c] = __shfl_sync(0xffffffffu, u[c % X], base + 2 * j + c / X);
                    p[c] = dr_pack2(uc[c], uc[c]);
                }
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const ulonglong2 kk = e2[j * D4 + DR_L * i];
#pragma unroll
                    for (int c = 0; c < VC; ++c) {
                        S[c][2 * i] = dr_fma2(kk.x, p[c], S[c][2 * i]);
                        S[c][2 * i + 1] = dr_fma2(kk.y, p[c], S[c][2 * i + 1]);
                    }
                }
#pragma unroll
                for (int x = 0; x < X; ++x) O[x] = fmaf(br[j], (l & 1) ? uc[X + x] : uc[x], O[x]);
            }
        }
        const int t = chunk * DR_C + my_t;
        float* row = out + (long)(first + t) * out_stride + (long)h * V + v0 + my_col;
#pragma unroll
        for (int x = 0; x < X; ++x)
            if (t < n_new && v0 + my_col + x < V) row[x] = O[x];
    }
#pragma unroll
    for (int c = 0; c < VC; ++c) {
        if (v0 + col0 + c >= V) continue;
#pragma unroll
        for (int i = 0; i < NI; ++i)
            if (l + DR_L * i < d4)
                reinterpret_cast<ulonglong2*>(st + (long)(v0 + col0 + c) * Dp)[l + DR_L * i] =
                    make_ulonglong2(S[c][2 * i], S[c][2 * i + 1]);
    }
}

// ------------------------------------------------------------------------------------- steps of one token a sequence
// The last products before the decays, the write strength and the gate of low rank, taken by the block that needs them
// (steps of few sequences: every block reads its head's rows of the weights).  Weights and rows are of the step's type; K
// counts are multiples of 8 and rows start on 16 bytes.  Null pointers: the product was taken before.
template <typename T>
struct DrDots {
    const T* h;                 // rows the mixer reads, with stride h_stride, width d
    long h_stride;
    int d;
    const T* wb;                // [H][d]
    const T* wa;                // [H][d]: one decay a head
    const T* wa2;               // [H * D][ra], read with the columns a_at.. of the projection
    const T* wg2;               // [H * V][rg], read with the columns g_at.. of the projection
    int ra, rg;
    long a_at, g_at;
};

__device__ __forceinline__ float dr_dot8(const float* __restrict__ w, const float* __restrict__ x) {
    const float4 a = *reinterpret_cast<const float4*>(w), b = *reinterpret_cast<const float4*>(w + 4);
    const float4 u = *reinterpret_cast<const float4*>(x), v = *reinterpret_cast<const float4*>(x + 4);
    return fmaf(a.x, u.x, fmaf(a.y, u.y, fmaf(a.z, u.z, fmaf(a.w, u.w, fmaf(b.x, v.x, fmaf(b.y, v.y, fmaf(b.z, v.z, b.w * v.w)))))));
}
__device__ __forceinline__ float dr_dot8(const __nv_bfloat16* __restrict__ w, const __nv_bfloat16* __restrict__ x) {
    const uint4 a = *reinterpret_cast<const uint4*>(w), b = *reinterpret_cast<const uint4*>(x);
    const __nv_bfloat162 *pa = reinterpret_cast<const __nv_bfloat162*>(&a), *pb = reinterpret_cast<const __nv_bfloat162*>(&b);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const float2 u = __bfloat1622float2(pa[i]), v = __bfloat1622float2(pb[i]);
        s = fmaf(u.x, v.x, s); s = fmaf(u.y, v.y, s);
    }
    return s;
}
// w . x over n elements by a warp; every lane gets the sum.
template <typename T>
__device__ __forceinline__ float dr_warp_dot(const T* __restrict__ w, const T* __restrict__ x, int n, int lane) {
    float s = 0.f;
#pragma unroll 4
    for (int i = lane * 8; i < n; i += 256) s += dr_dot8(w + i, x + i);
    return warp_sum(s);
}
// The same by four neighbouring lanes (part 0..3), for short rows.
template <typename T>
__device__ __forceinline__ float dr_quad_dot(const T* __restrict__ w, const T* __restrict__ x, int n, int part) {
    float s = 0.f;
#pragma unroll 4
    for (int i = part * 8; i < n; i += 32) s += dr_dot8(w + i, x + i);
    s += __shfl_xor_sync(0xffffffffu, s, 1);
    return s + __shfl_xor_sync(0xffffffffu, s, 2);
}

// grid (heads, sequences); blockDim a multiple of 32.  norm_w: [V]; gate rows with stride gate_stride ([H * V] numbers,
// null: none), gate_kind 1 sigmoid, 2 silu; out rows with stride out_stride.
template <typename T, int L, int NI, bool CH>
__global__ void __launch_bounds__(NI > 4 ? 512 : 1024)
dr_decode_kernel(DrIn<T> in, DrDots<T> dots, float* __restrict__ state, const float* __restrict__ norm_w, float eps,
                 const T* __restrict__ gate, long gate_stride, int gate_kind, T* __restrict__ out, long out_stride) {
    constexpr int DS = 4 * L * NI;
    extern __shared__ __align__(16) float dr_sm[];
    float* q_s = dr_sm;                                    // [DS]
    float* k_s = q_s + DS;                                 // [DS]
    float* g_s = k_s + DS;                                 // [DS] (CH: the decays; else one number)
    float* v_s = g_s + DS;                                 // [V]
    float* o_s = v_s + in.V;                               // [V]
    float* gate_s = o_s + in.V;                            // [V] where dots.wg2 is given
    __shared__ float scratch[33], scale_s[2], beta_s;
    pdl_launch_dependents();
    const int h = blockIdx.x, b = blockIdx.y;
    const int tid = threadIdx.x, l = tid % L, cols = blockDim.x / L;
    const int kv = h / (in.H / in.G), d4 = in.Dp / 4;
    const int slot = in.slots[b], pos = in.past_lens[b];
    float4* st = reinterpret_cast<float4*>(state + ((long)slot * in.H + h) * in.V * in.Dp);
    // this thread's part of the first columns: nothing of the step but this block writes it
    float4 S[NI];
    int vcol = tid / L;
#pragma unroll
    for (int i = 0; i < NI; ++i)
        S[i] = (vcol < in.V && l + L * i < d4) ? st[(long)vcol * d4 + l + L * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_wait();
    const T* x = in.proj + (long)b * in.proj_stride;
    float* ring = in.ring + (long)slot * in.K * in.C;
    float* ring_row = ring + (long)(pos % in.K) * in.C;
    for (int i = tid; i < 2 * DS; i += blockDim.x) {
        const int d = i < DS ? i : i - DS;
        const int c = (i < DS ? kv : in.G + kv) * in.D + d;
        float y = 0.f;
        if (d < in.D) {
            y = dr_silu(dr_conv1<T>(in, x, ring, 0, pos, c));
            ring_row[c] = to_float(x[c]);                  // heads of a group write the same numbers
        }
        q_s[i] = y;                                        // k_s lies behind q_s
    }
    for (int i = tid; i < in.V; i += blockDim.x) {
        const int c = 2 * in.G * in.D + h * in.V + i;
        v_s[i] = dr_silu(dr_conv1<T>(in, x, ring, 0, pos, c));
        ring_row[c] = to_float(x[c]);
    }
    // decays and the write strength; the last warps, which have no part in the convolution of short heads, come first
    const float rate = in.rate[h];
    const int warp = tid >> 5, lane = tid & 31, n_warps = blockDim.x >> 5;
    if (warp == n_warps - 1) {
        const float z = dots.wb != nullptr ? dr_warp_dot<T>(dots.wb + (long)h * dots.d, dots.h + (long)b * dots.h_stride, dots.d, lane)
                                           : in.b[(long)b * in.b_stride + h];
        if (lane == 0) beta_s = dr_sigmoid(z);
    }
    if (!CH && warp == n_warps - 2) {
        const float z = dots.wa != nullptr ? dr_warp_dot<T>(dots.wa + (long)h * dots.d, dots.h + (long)b * dots.h_stride, dots.d, lane)
                                           : in.a[(long)b * in.a_stride + h];
        if (lane == 0) g_s[0] = expf(-rate * dr_softplus(z + in.dt_bias[h]));
    }
    if constexpr (CH) {
        if (dots.wa2 != nullptr) {
            for (int i0 = 0; i0 < DS; i0 += blockDim.x / 4) {          // the same number of rounds for every thread
                const int i = i0 + tid / 4, row = min(i, in.D - 1);
                const float z = dr_quad_dot<T>(dots.wa2 + ((long)h * in.D + row) * dots.ra, x + dots.a_at, dots.ra, tid & 3);
                if ((tid & 3) == 0 && i < DS)
                    g_s[i] = i < in.D ? expf(-rate * dr_softplus(z + in.dt_bias[h * in.D + i])) : 0.f;
            }
        } else {
            for (int i = tid; i < DS; i += blockDim.x)
                g_s[i] = i < in.D ? expf(-rate * dr_softplus(in.a[(long)b * in.a_stride + (long)h * in.D + i] + in.dt_bias[h * in.D + i])) : 0.f;
        }
    }
    if (dots.wg2 != nullptr) {
        for (int i0 = 0; i0 < in.V; i0 += blockDim.x / 4) {
            const int i = i0 + tid / 4, row = min(i, in.V - 1);
            const float z = dr_quad_dot<T>(dots.wg2 + ((long)h * in.V + row) * dots.rg, x + dots.g_at, dots.rg, tid & 3);
            if ((tid & 3) == 0 && i < in.V) gate_s[i] = z;
        }
    }
    __syncthreads();
    if (tid < 64) {
        const float* r = tid < 32 ? q_s : k_s;
        float ss = 0.f;
        for (int i = tid & 31; i < DS; i += 32) ss = fmaf(r[i], r[i], ss);
        ss = warp_sum(ss);
        if ((tid & 31) == 0) scale_s[tid >> 5] = (tid < 32 ? 1.0f / sqrtf((float)in.D) : 1.0f) / sqrtf(ss + 1e-6f);
    }
    __syncthreads();
    for (int i = tid; i < 2 * DS; i += blockDim.x) q_s[i] *= scale_s[i < DS ? 0 : 1];
    __syncthreads();
    const float4* q4 = reinterpret_cast<const float4*>(q_s);
    const float4* k4 = reinterpret_cast<const float4*>(k_s);
    const float4* g4 = reinterpret_cast<const float4*>(g_s);
    const float g1 = CH ? 0.f : g_s[0], bt = beta_s;
    float ss = 0.f;
    for (int v0 = 0; v0 < in.V; v0 += cols) {              // the same number of rounds for every thread: shuffles inside
        vcol = v0 + tid / L;
        const bool live = vcol < in.V;
        if (v0 > 0) {
#pragma unroll
            for (int i = 0; i < NI; ++i)
                S[i] = (live && l + L * i < d4) ? st[(long)vcol * d4 + l + L * i] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float p0 = 0.f, p1 = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 kk = k4[l + L * i];
            float4 gg = make_float4(g1, g1, g1, g1);
            if constexpr (CH) gg = g4[l + L * i];
            S[i].x *= gg.x; S[i].y *= gg.y; S[i].z *= gg.z; S[i].w *= gg.w;
            p0 = fmaf(kk.x, S[i].x, p0); p1 = fmaf(kk.y, S[i].y, p1); p0 = fmaf(kk.z, S[i].z, p0); p1 = fmaf(kk.w, S[i].w, p1);
        }
        const float u = bt * ((live ? v_s[vcol] : 0.f) - dr_sum<L>(p0 + p1));
        float o0 = 0.f, o1 = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 kk = k4[l + L * i], qq = q4[l + L * i];
            S[i].x = fmaf(kk.x, u, S[i].x); S[i].y = fmaf(kk.y, u, S[i].y);
            S[i].z = fmaf(kk.z, u, S[i].z); S[i].w = fmaf(kk.w, u, S[i].w);
            o0 = fmaf(qq.x, S[i].x, o0); o1 = fmaf(qq.y, S[i].y, o1); o0 = fmaf(qq.z, S[i].z, o0); o1 = fmaf(qq.w, S[i].w, o1);
            if (live && l + L * i < d4) st[(long)vcol * d4 + l + L * i] = S[i];
        }
        const float o = dr_sum<L>(o0 + o1);
        if (live && l == 0) { o_s[vcol] = o; ss = fmaf(o, o, ss); }
    }
    ss = block_sum(ss, scratch);                           // synchronises: o_s is complete behind it
    const float inv = 1.0f / sqrtf(ss / (float)in.V + eps);
    for (int i = tid; i < in.V; i += blockDim.x) {
        float y = o_s[i] * inv * norm_w[i];
        if (gate_kind != 0) {
            const float gv = dots.wg2 != nullptr ? gate_s[i] : to_float(gate[(long)b * gate_stride + (long)h * in.V + i]);
            const float sg = dr_sigmoid(gv);
            y *= gate_kind == 2 ? gv * sg : sg;
        }
        out[(long)b * out_stride + (long)h * in.V + i] = from_float<T>(y);
    }
}

// The (L, NI) a key size runs with: the smallest 4 L NI that holds it.
static inline bool dr_shape(int Dp, int& L, int& NI) {
    L = 8;
    for (int ni : {1, 2, 3, 4, 6, 8})
        if (4 * 8 * ni >= Dp) { NI = ni; return true; }
    L = 32;
    NI = 4;
    return 4 * 32 * NI >= Dp;
}

}  // namespace zlm

using namespace zlm;

#define ZLM_DR_SHAPES(F)                                                                                              \
    if (L == 8) {                                                                                                     \
        switch (NI) {                                                                                                 \
            case 1: F(8, 1); break;                                                                                   \
            case 2: F(8, 2); break;                                                                                   \
            case 3: F(8, 3); break;                                                                                   \
            case 4: F(8, 4); break;                                                                                   \
            case 6: F(8, 6); break;                                                                                   \
            default: F(8, 8); break;                                                                                  \
        }                                                                                                             \
    } else {                                                                                                          \
        F(32, 4);                                                                                                     \
    }

template <typename T>
static int dr_fill(DrIn<T>& in, const void* proj, long proj_stride, const float* taps, float* ring, int H, int G, int D, int V,
                   int K, const float* a, long a_stride, const float* b, long b_stride, const float* rate,
                   const float* dt_bias, const int* slots, const int* past_lens, const int* cu_seqlens) {
    if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0 || K <= 0) return ZLM_ERR_BAD_ARG;
    in.proj = (const T*)proj; in.proj_stride = proj_stride; in.taps = taps; in.ring = ring;
    in.H = H; in.G = G; in.D = D; in.V = V; in.C = 2 * G * D + H * V; in.K = K;
    in.Dp = (D + 3) / 4 * 4; in.Vp = (V + 3) / 4 * 4;
    in.a = a; in.a_stride = a_stride; in.b = b; in.b_stride = b_stride; in.rate = rate; in.dt_bias = dt_bias;
    in.slots = slots; in.past_lens = past_lens; in.cu_seqlens = cu_seqlens;
    return 0;
}

template <typename T>
static int dr_prep_launch(const DrIn<T>& in, int channel_decay, int n_seqs, int max_new, float* qk, float* v, float* g,
                          float* beta, cudaStream_t stream) {
    const int tile = in.K - 1 > 8 ? in.K - 1 : 8;
    const int units = 2 * in.G + 2 * in.H;
    dim3 grid((max_new + tile - 1) / tile, (units + DR_PREP_WARPS - 1) / DR_PREP_WARPS, n_seqs);
    if (grid.y > 65535 || grid.z > 65535) return ZLM_ERR_UNSUPPORTED;
    const size_t smem = (size_t)DR_PREP_WARPS * in.Dp * sizeof(float);
    const bool vec = in.D % 4 == 0 && in.V % 4 == 0 && in.proj_stride % 4 == 0 && (uintptr_t)in.proj % 16 == 0 &&
                     (uintptr_t)in.taps % 16 == 0 && (uintptr_t)in.ring % 16 == 0;
    cudaError_t e = vec ? launch_pdl(dr_prep_kernel<T, true>, grid, dim3(DR_PREP_WARPS * 32), smem, stream, in, channel_decay,
                                     tile, qk, v, g, beta)
                        : launch_pdl(dr_prep_kernel<T, false>, grid, dim3(DR_PREP_WARPS * 32), smem, stream, in, channel_decay,
                                     tile, qk, v, g, beta);
    return e == cudaSuccess ? launch_status() : (int)e;
}

// proj: rows whose first 2 G D + H V columns are q | k | v; a: float rows of H (or H D, channel_decay) numbers, b of H.
// qk: float [T][2 G][Dp], v: [T][H][Vp], g: [T][H][Dp] or [T][H], beta: [T][H], with Dp and Vp rounded up to fours.
ZLM_EXPORT int zlm_delta_prep(const void* proj, int dtype, long proj_stride, const float* taps, float* ring, int H, int G,
                              int D, int V, int K, const float* a, long a_stride, int channel_decay, const float* b,
                              long b_stride, const float* rate, const float* dt_bias, const int* slots,
                              const int* past_lens, const int* cu_seqlens, int n_seqs, int max_new, float* qk, float* v,
                              float* g, float* beta, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return 0;
    if (dtype == ZLM_F32) {
        DrIn<float> in;
        const int s = dr_fill<float>(in, proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, b, b_stride, rate, dt_bias,
                                     slots, past_lens, cu_seqlens);
        return s ? s : dr_prep_launch<float>(in, channel_decay, n_seqs, max_new, qk, v, g, beta, stream);
    }
    if (dtype == ZLM_BF16) {
        DrIn<__nv_bfloat16> in;
        const int s = dr_fill<__nv_bfloat16>(in, proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, b, b_stride, rate,
                                             dt_bias, slots, past_lens, cu_seqlens);
        return s ? s : dr_prep_launch<__nv_bfloat16>(in, channel_decay, n_seqs, max_new, qk, v, g, beta, stream);
    }
    return ZLM_ERR_UNSUPPORTED;
}

// The float4 a lane of DR_L holds of a row of Dp elements, or 0: too long.
static inline int dr_scan_ni(int Dp) {
    for (int ni : {1, 2, 3, 4, 8})
        if (4 * DR_L * ni >= Dp) return ni;
    return 0;
}

#define ZLM_DR_NI(F)                                                                                                   \
    switch (ni) {                                                                                                      \
        case 1: F(1); break;                                                                                           \
        case 2: F(2); break;                                                                                           \
        case 3: F(3); break;                                                                                           \
        case 4: F(4); break;                                                                                           \
        default: F(8); break;                                                                                          \
    }
// Launch kernel k with smem bytes of shared memory, raising its limit once.
#define ZLM_DR_RAISED(k, which, grid, ...)                                                                             \
    do {                                                                                                               \
        static size_t raised[2] = {40 * 1024, 40 * 1024};                                                              \
        if (raised[which] < smem) {                                                                                    \
            e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                       \
            if (e != cudaSuccess) return (int)e;                                                                       \
            raised[which] = smem;                                                                                      \
        }                                                                                                              \
        e = launch_pdl(k, grid, dim3(threads), smem, stream, __VA_ARGS__);                                             \
    } while (0)

// What every chunk contributes apart from the state: rec, float [zlm_delta_chunks][H][zlm_delta_record] (dr_chunk_kernel).
// g: [T][H][Dp] (channel_decay) or [T][H].
ZLM_EXPORT int zlm_delta_chunk(const float* qk, const float* g, int channel_decay, const float* beta, const int* cu_seqlens,
                               float* rec, int n_seqs, int max_new, int H, int G, int D, cudaStream_t stream) {
    if (n_seqs <= 0 || max_new <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0) return ZLM_ERR_BAD_ARG;
    const int Dp = (D + 3) / 4 * 4, ni = dr_scan_ni(Dp), which = channel_decay ? 1 : 0;
    if (ni == 0 || H > 65535 || n_seqs > 65535) return ZLM_ERR_UNSUPPORTED;
    const size_t smem = (size_t)DR_C * 64 * ni * (which ? 3 : 2) * sizeof(float);
    dim3 grid((max_new + DR_C - 1) / DR_C, H, n_seqs);
    const int threads = DR_THREADS;
    cudaError_t e = cudaSuccess;
#define ZLM_DR_CHUNK(NN)                                                                                               \
    do {                                                                                                               \
        auto* k = which ? dr_chunk_kernel<NN, true> : dr_chunk_kernel<NN, false>;                                      \
        ZLM_DR_RAISED(k, which, grid, qk, g, beta, cu_seqlens, rec, H, G, Dp);                                         \
    } while (0)
    ZLM_DR_NI(ZLM_DR_CHUNK)
#undef ZLM_DR_CHUNK
    return e == cudaSuccess ? launch_status() : (int)e;
}

// The most chunks a step of T tokens of n_seqs sequences can have, and the floats of a record for keys of D elements (0: too
// long).
ZLM_EXPORT int zlm_delta_chunks(int T, int n_seqs) { return T / DR_C + n_seqs + 1; }
ZLM_EXPORT int zlm_delta_record(int D) {
    const int ni = dr_scan_ni((D + 3) / 4 * 4);
    return ni ? dr_record(ni) : 0;
}

// state: float [slots][H][V][Dp]; v: [T][H][Vp]; out: float rows of H V numbers.
ZLM_EXPORT int zlm_delta_scan(const float* rec, const float* v, float* state, const int* slots, const int* cu_seqlens,
                              float* out, long out_stride, int n_seqs, int H, int D, int V, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || D <= 0 || V <= 0) return ZLM_ERR_BAD_ARG;
    const int Dp = (D + 3) / 4 * 4, Vp = (V + 3) / 4 * 4, ni = dr_scan_ni(Dp);
    if (ni == 0 || H > 65535 || n_seqs > 65535) return ZLM_ERR_UNSUPPORTED;
    dim3 grid((V + DR_VT - 1) / DR_VT, H, n_seqs);
    const size_t smem = (size_t)DR_STAGES * dr_stage(ni) * sizeof(float);
    // a block an SM at most: more warps hide more of each other's waits; else the SM's shared memory sets the pace
    const bool few = (long)grid.x * grid.y * grid.z <= 148;
    cudaError_t e = cudaSuccess;
#define ZLM_DR_SCAN(NN)                                                                                                \
    do {                                                                                                               \
        constexpr int WIDE = NN <= 4 ? 4 : 2;            /* the registers of longer columns */                         \
        const int which = few ? 0 : 1, threads = dr_scan_threads(few ? 2 : WIDE);                                      \
        auto* k = few ? dr_scan_kernel<NN, 2> : dr_scan_kernel<NN, WIDE>;                                              \
        ZLM_DR_RAISED(k, which, grid, rec, v, state, slots, cu_seqlens, out, out_stride, H, Dp, V, Vp);                \
    } while (0)
    ZLM_DR_NI(ZLM_DR_SCAN)
#undef ZLM_DR_SCAN
    return e == cudaSuccess ? launch_status() : (int)e;
}

template <typename T>
static int dr_decode_launch(const DrIn<T>& in, const DrDots<T>& dots, int channel_decay, int n_seqs, float* state, const float* norm_w, float eps,
                            const void* gate, long gate_stride, int gate_kind, void* out, long out_stride,
                            cudaStream_t stream) {
    int L, NI;
    if (!dr_shape(in.Dp, L, NI) || n_seqs > 65535) return ZLM_ERR_UNSUPPORTED;
    int threads = (in.V * L + 31) / 32 * 32;
    threads = threads < 64 ? 64 : (threads > 1024 ? 1024 : threads);
    if (NI > 4 && threads > 512) threads = 512;
    const size_t smem = ((size_t)3 * 4 * L * NI + 3 * in.V) * sizeof(float);
    if (smem > 48 * 1024) return ZLM_ERR_UNSUPPORTED;
    dim3 grid(in.H, n_seqs);
    cudaError_t e = cudaSuccess;
#define ZLM_DR_DEC(LL, NN)                                                                                             \
    do {                                                                                                               \
        auto* k = channel_decay ? dr_decode_kernel<T, LL, NN, true> : dr_decode_kernel<T, LL, NN, false>;              \
        e = launch_pdl(k, grid, dim3(threads), smem, stream, in, dots, state, norm_w, eps, (const T*)gate, gate_stride, gate_kind, \
                       (T*)out, out_stride);                                                                           \
    } while (0)
    ZLM_DR_SHAPES(ZLM_DR_DEC)
#undef ZLM_DR_DEC
    return e == cudaSuccess ? launch_status() : (int)e;
}

template <typename T>
static int dr_decode_typed(const void* proj, long proj_stride, const float* taps, float* ring, int H, int G, int D, int V, int K,
                           const float* a, long a_stride, int channel_decay, const float* b, long b_stride, const float* rate,
                           const float* dt_bias, const int* slots, const int* past_lens, int n_seqs, float* state,
                           const float* norm_w, float eps, const void* gate, long gate_stride, int gate_kind, const void* h,
                           long h_stride, int d, const void* wb, const void* wa, const void* wa2, int ra, long a_at,
                           const void* wg2, int rg, long g_at, void* out, long out_stride, cudaStream_t stream) {
    DrIn<T> in;
    const int s = dr_fill<T>(in, proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, b, b_stride, rate, dt_bias, slots,
                             past_lens, nullptr);
    if (s) return s;
    const int per16 = 16 / (int)sizeof(T);
    if ((wb == nullptr && b == nullptr) || (gate_kind != 0 && gate == nullptr && wg2 == nullptr) ||
        (channel_decay ? (a == nullptr && wa2 == nullptr) : (a == nullptr && wa == nullptr)) ||
        ((wb != nullptr || wa != nullptr) && (h == nullptr || d % 8 || h_stride % per16)) ||
        (wa2 != nullptr && (ra % 8 || a_at % per16 || proj_stride % per16)) ||
        (wg2 != nullptr && (rg % 8 || g_at % per16 || proj_stride % per16)))
        return ZLM_ERR_BAD_ARG;
    for (const void* p : {h, wb, wa, wa2, wg2, wa2 || wg2 ? proj : nullptr})
        if ((uintptr_t)p % 16) return ZLM_ERR_BAD_ARG;
    DrDots<T> dots;
    dots.h = (const T*)h; dots.h_stride = h_stride; dots.d = d; dots.wb = (const T*)wb; dots.wa = (const T*)wa;
    dots.wa2 = (const T*)wa2; dots.wg2 = (const T*)wg2; dots.ra = ra; dots.rg = rg; dots.a_at = a_at; dots.g_at = g_at;
    return dr_decode_launch<T>(in, dots, channel_decay, n_seqs, state, norm_w, eps, gate, gate_stride, gate_kind, out, out_stride,
                               stream);
}

// One token a sequence (row b of proj belongs to sequence b).  gate: rows of H V numbers of proj's type, or null;
// gate_kind 0 none, 1 sigmoid, 2 silu; norm_w: float [V]; out: rows of H V numbers of proj's type.  The products behind b, a
// and gate may be left to the kernel (DrDots): wb [H][d] and wa [H][d] with the rows h; wa2 [H D][ra] with the columns from
// a_at on of proj, wg2 [H V][rg] with those from g_at on.
ZLM_EXPORT int zlm_delta_decode(const void* proj, int dtype, long proj_stride, const float* taps, float* ring, int H, int G,
                                int D, int V, int K, const float* a, long a_stride, int channel_decay, const float* b,
                                long b_stride, const float* rate, const float* dt_bias, const int* slots,
                                const int* past_lens, int n_seqs, float* state, const float* norm_w, float eps,
                                const void* gate, long gate_stride, int gate_kind, const void* h, long h_stride, int d,
                                const void* wb, const void* wa, const void* wa2, int ra, long a_at, const void* wg2, int rg,
                                long g_at, void* out, long out_stride, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    auto run = dtype == ZLM_F32 ? dr_decode_typed<float> : dtype == ZLM_BF16 ? dr_decode_typed<__nv_bfloat16> : nullptr;
    if (run == nullptr) return ZLM_ERR_UNSUPPORTED;
    return run(proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, channel_decay, b, b_stride, rate, dt_bias, slots,
               past_lens, n_seqs, state, norm_w, eps, gate, gate_stride, gate_kind, h, h_stride, d, wb, wa, wa2, ra, a_at, wg2, rg,
               g_at, out, out_stride, stream);
}
