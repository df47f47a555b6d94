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
// Any other step is two kernels.  dr_prep makes q, k, v, g, beta of every token in float and writes the ring.  dr_scan
// walks a sequence's tokens with S in registers: a column of S is spread over L lanes of a warp (4 NI elements a lane)
// and the columns of a head over blocks, which need nothing from each other.  A token would cost two dependent
// reductions over those lanes; the walk keeps the write of the token before pending instead,
//     Sbar_t = diag(g_t) (Sbar_(t-1) + k_(t-1) u_(t-1)),     u_t = beta_t (v_t - r_t - c_t u_(t-1)),
//     r_(t+1) = (g_(t+1) k_(t+1)) . Sbar_t,  c_t = (g_t k_t) . k_(t-1),   o_t = q_t . Sbar_t + (q_t . k_t) u_t,
// so the reduction that u_(t+1) needs starts before u_t is known, and both reductions of a token run side by side.
// Tokens come in chunks through shared memory (cp.async, two stages); c and q . k are taken once a chunk.  Every sum is
// float FMA; nothing that enters the recurrence passes through a 16-bit type behind the projection.
#include "common.cuh"

namespace zlm {

constexpr int DR_THREADS = 128;      // of the scan: 128 / L value columns a block
constexpr int DR_PREP_WARPS = 4;

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
    pdl_launch_dependents();
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
            if (channel_decay) {
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
    for (int i = lo; i < hi; ++i) {
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

__host__ __device__ constexpr int dr_chunk(int DS) { return 2048 / DS > 16 ? 16 : 2048 / DS; }      // tokens of a chunk
static inline size_t dr_scan_floats(int L, int NI, bool ch) {
    const int DS = 4 * L * NI, TC = dr_chunk(DS), VT = DR_THREADS / L;
    const size_t stage = (size_t)TC * ((ch ? 3 : 2) * DS + VT + (ch ? 1 : 2));
    return 2 * ((stage + 3) / 4 * 4) + (ch ? (size_t)TC * DS : 0) + 2 * TC + (size_t)TC * VT;
}

// grid (value tiles, heads, sequences).  qk: float [T][2 G][Dp], v: [T][H][Vp], g: [T][H][Dp] or [T][H], beta: [T][H];
// out: float [T][H * V] rows.
template <int L, int NI, bool CH>
__global__ void __launch_bounds__(DR_THREADS)
dr_scan_kernel(const float* __restrict__ qk, const float* __restrict__ v, const float* __restrict__ g,
               const float* __restrict__ beta, float* __restrict__ state, const int* __restrict__ slots,
               const int* __restrict__ cu_seqlens, float* __restrict__ out, long out_stride, int H, int G, int Dp, int V,
               int Vp) {
    constexpr int DS = 4 * L * NI, TC = dr_chunk(DS), VT = DR_THREADS / L, D4 = DS / 4;
    constexpr int STAGE = (TC * ((CH ? 3 : 2) * DS + VT + (CH ? 1 : 2)) + 3) / 4 * 4;
    extern __shared__ __align__(16) float dr_sm[];
    float* kg_s = dr_sm + 2 * STAGE;                       // [TC][DS] g k (CH)
    float* c_s = kg_s + (CH ? TC * DS : 0);                // [TC]
    float* qd_s = c_s + TC;                                // [TC]
    float* o_s = qd_s + TC;                                // [TC][VT]
    pdl_launch_dependents();
    const int tid = threadIdx.x, l = tid % L, col = tid / L;
    const int b = blockIdx.z, h = blockIdx.y, v0 = blockIdx.x * VT;
    const int kv = h / (H / G);
    const int d4 = Dp / 4;
    const int vcol = v0 + col;
    const bool live = vcol < V;
    // what stands behind the live elements of a row stays zero
    for (int i = tid; i < 2 * STAGE; i += DR_THREADS) dr_sm[i] = 0.f;
    if constexpr (CH) for (int i = tid; i < TC * DS; i += DR_THREADS) kg_s[i] = 0.f;
    float* st = state + (((long)slots[b] * H + h) * V + (live ? vcol : 0)) * Dp;
    float4 S[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i)
        S[i] = (live && l + L * i < d4) ? reinterpret_cast<const float4*>(st)[l + L * i] : make_float4(0.f, 0.f, 0.f, 0.f);
    pdl_wait();
    __syncthreads();
    const int first = cu_seqlens[b], n_new = cu_seqlens[b + 1] - first;
    auto fetch = [&](int at, int stage) {
        float* sm = dr_sm + stage * STAGE;
        const int n = min(TC, n_new - at);
        for (int idx = tid; idx < n * d4; idx += DR_THREADS) {
            const int j = idx / d4, i = idx - j * d4;
            const long t = first + at + j;
            dr_cp16(sm + j * DS + 4 * i, qk + (t * 2 * G + kv) * Dp + 4 * i);
            dr_cp16(sm + (TC + j) * DS + 4 * i, qk + (t * 2 * G + G + kv) * Dp + 4 * i);
            if constexpr (CH) dr_cp16(sm + (2 * TC + j) * DS + 4 * i, g + (t * H + h) * Dp + 4 * i);
        }
        float* v_s = sm + (CH ? 3 : 2) * TC * DS;
        for (int idx = tid; idx < n * (VT / 4); idx += DR_THREADS) {
            const int j = idx / (VT / 4), i = idx - j * (VT / 4);
            if (v0 + 4 * i < Vp) dr_cp16(v_s + j * VT + 4 * i, v + ((first + at + j) * (long)H + h) * Vp + v0 + 4 * i);
        }
        float* s_s = v_s + TC * VT;
        for (int j = tid; j < n; j += DR_THREADS) {
            const long t = first + at + j;
            s_s[j] = beta[t * H + h];
            if constexpr (!CH) s_s[TC + j] = g[t * H + h];
        }
        dr_cp_commit();
    };
    fetch(0, 0);
    for (int at = 0, stage = 0; at < n_new; at += TC, stage ^= 1) {
        const int n = min(TC, n_new - at);
        if (at + TC < n_new) { fetch(at + TC, stage ^ 1); dr_cp_wait<1>(); } else { dr_cp_wait<0>(); }
        __syncthreads();
        const float4* q4 = reinterpret_cast<const float4*>(dr_sm + stage * STAGE);
        const float4* k4 = q4 + TC * D4;
        const float4* g4 = k4 + TC * D4;                   // CH
        const float* v_s = dr_sm + stage * STAGE + (CH ? 3 : 2) * TC * DS;
        const float* b_s = v_s + TC * VT;
        const float* g_s = b_s + TC;                       // !CH
        const float4* kg4 = CH ? reinterpret_cast<const float4*>(kg_s) : k4;
        // q . k of a token, (g k) . k of the token before, and g k
        for (int t0 = 0; t0 < n; t0 += VT) {
            const int t = t0 + col;
            float qd = 0.f, cc = 0.f;
            if (t < n) {
#pragma unroll
                for (int i = 0; i < NI; ++i) {
                    const float4 kk = k4[t * D4 + l + L * i], qq = q4[t * D4 + l + L * i];
                    float4 kg = kk;
                    if constexpr (CH) {
                        const float4 gg = g4[t * D4 + l + L * i];
                        kg = make_float4(kk.x * gg.x, kk.y * gg.y, kk.z * gg.z, kk.w * gg.w);
                        reinterpret_cast<float4*>(kg_s)[t * D4 + l + L * i] = kg;
                    }
                    qd = fmaf(qq.x, kk.x, qd); qd = fmaf(qq.y, kk.y, qd); qd = fmaf(qq.z, kk.z, qd); qd = fmaf(qq.w, kk.w, qd);
                    if (t > 0) {
                        const float4 kp = k4[(t - 1) * D4 + l + L * i];
                        cc = fmaf(kg.x, kp.x, cc); cc = fmaf(kg.y, kp.y, cc); cc = fmaf(kg.z, kp.z, cc); cc = fmaf(kg.w, kp.w, cc);
                    }
                }
            }
            qd = dr_sum<L>(qd);
            cc = dr_sum<L>(cc);
            if (t < n && l == 0) {
                qd_s[t] = qd;
                c_s[t] = CH ? cc : cc * g_s[t];
            }
        }
        __syncthreads();
        float r, u = 0.f;
        {
            float p0 = 0.f, p1 = 0.f;
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float4 kk = kg4[l + L * i];
                p0 = fmaf(kk.x, S[i].x, p0); p1 = fmaf(kk.y, S[i].y, p1);
                p0 = fmaf(kk.z, S[i].z, p0); p1 = fmaf(kk.w, S[i].w, p1);
            }
            r = dr_sum<L>(p0 + p1);
            if constexpr (!CH) r *= g_s[0];
        }
        for (int t = 0; t < n; ++t) {
            float o0 = 0.f, o1 = 0.f, p0 = 0.f, p1 = 0.f;
            const int tn = t + 1 < n ? t + 1 : t, tp = t > 0 ? t - 1 : 0;        // u is zero where there is no token before
            const float gt = CH ? 0.f : g_s[t];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                const float4 kp = k4[tp * D4 + l + L * i];
                float4 s = S[i];
                s.x = fmaf(kp.x, u, s.x); s.y = fmaf(kp.y, u, s.y); s.z = fmaf(kp.z, u, s.z); s.w = fmaf(kp.w, u, s.w);
                if constexpr (CH) {
                    const float4 gg = g4[t * D4 + l + L * i];
                    s.x *= gg.x; s.y *= gg.y; s.z *= gg.z; s.w *= gg.w;
                } else {
                    s.x *= gt; s.y *= gt; s.z *= gt; s.w *= gt;
                }
                S[i] = s;
                const float4 kn = kg4[tn * D4 + l + L * i], qq = q4[t * D4 + l + L * i];
                p0 = fmaf(kn.x, s.x, p0); p1 = fmaf(kn.y, s.y, p1); p0 = fmaf(kn.z, s.z, p0); p1 = fmaf(kn.w, s.w, p1);
                o0 = fmaf(qq.x, s.x, o0); o1 = fmaf(qq.y, s.y, o1); o0 = fmaf(qq.z, s.z, o0); o1 = fmaf(qq.w, s.w, o1);
            }
            u = b_s[t] * (v_s[t * VT + col] - fmaf(c_s[t], u, r));
            r = dr_sum<L>(p0 + p1);
            if constexpr (!CH) r *= g_s[tn];
            const float o = fmaf(qd_s[t], u, dr_sum<L>(o0 + o1));
            if (l == 0) o_s[t * VT + col] = o;
        }
        // the last token's write
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 kp = k4[(n - 1) * D4 + l + L * i];
            S[i].x = fmaf(kp.x, u, S[i].x); S[i].y = fmaf(kp.y, u, S[i].y);
            S[i].z = fmaf(kp.z, u, S[i].z); S[i].w = fmaf(kp.w, u, S[i].w);
        }
        __syncthreads();
        for (int idx = tid; idx < n * VT; idx += DR_THREADS) {
            const int j = idx / VT, c = idx - j * VT;
            if (v0 + c < V) out[(long)(first + at + j) * out_stride + (long)h * V + v0 + c] = o_s[idx];
        }
    }
    if (live) {
#pragma unroll
        for (int i = 0; i < NI; ++i)
            if (l + L * i < d4) reinterpret_cast<float4*>(st)[l + L * i] = S[i];
    }
}

// ------------------------------------------------------------------------------------- steps of one token a sequence
// grid (heads, sequences); blockDim a multiple of 32.  norm_w: [V]; gate rows with stride gate_stride ([H * V] numbers,
// null: none), gate_kind 1 sigmoid, 2 silu; out rows with stride out_stride.
template <typename T, int L, int NI, bool CH>
__global__ void __launch_bounds__(NI > 4 ? 512 : 1024)
dr_decode_kernel(DrIn<T> in, float* __restrict__ state, const float* __restrict__ norm_w, float eps,
                 const T* __restrict__ gate, long gate_stride, int gate_kind, T* __restrict__ out, long out_stride) {
    constexpr int DS = 4 * L * NI;
    extern __shared__ __align__(16) float dr_sm[];
    float* q_s = dr_sm;                                    // [DS]
    float* k_s = q_s + DS;                                 // [DS]
    float* g_s = k_s + DS;                                 // [DS] (CH: the decays; else one number)
    float* v_s = g_s + DS;                                 // [V]
    float* o_s = v_s + in.V;                               // [V]
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
    const float rate = in.rate[h];
    if constexpr (CH) {
        for (int i = tid; i < DS; i += blockDim.x)
            g_s[i] = i < in.D ? expf(-rate * dr_softplus(in.a[(long)b * in.a_stride + (long)h * in.D + i] + in.dt_bias[h * in.D + i])) : 0.f;
    } else if (tid == 0) {
        g_s[0] = expf(-rate * dr_softplus(in.a[(long)b * in.a_stride + h] + in.dt_bias[h]));
    }
    if (tid == 0) beta_s = dr_sigmoid(in.b[(long)b * in.b_stride + h]);
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
        if (gate != nullptr) {
            const float gv = to_float(gate[(long)b * gate_stride + (long)h * in.V + i]);
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
    for (int ni : {4, 8})
        if (4 * 32 * ni >= Dp) { NI = ni; return true; }
    return false;
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
        switch (NI) {                                                                                                 \
            case 4: F(32, 4); break;                                                                                  \
            default: F(32, 8); break;                                                                                 \
        }                                                                                                             \
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

// state: float [slots][H][V][Dp]; out: float rows of H V numbers.
ZLM_EXPORT int zlm_delta_scan(const float* qk, const float* v, const float* g, int channel_decay, const float* beta,
                              float* state, const int* slots, const int* cu_seqlens, float* out, long out_stride, int n_seqs,
                              int H, int G, int D, int V, cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || V <= 0) return ZLM_ERR_BAD_ARG;
    const int Dp = (D + 3) / 4 * 4, Vp = (V + 3) / 4 * 4;
    int L, NI;
    if (!dr_shape(Dp, L, NI) || H > 65535 || n_seqs > 65535) return ZLM_ERR_UNSUPPORTED;
    const int VT = DR_THREADS / L;
    dim3 grid((V + VT - 1) / VT, H, n_seqs);
    const size_t smem = dr_scan_floats(L, NI, channel_decay != 0) * sizeof(float);
    cudaError_t e = cudaSuccess;
#define ZLM_DR_SCAN(LL, NN)                                                                                            \
    do {                                                                                                               \
        auto* k = channel_decay ? dr_scan_kernel<LL, NN, true> : dr_scan_kernel<LL, NN, false>;                        \
        static size_t raised[2] = {0, 0};                                                                              \
        if (smem > 48 * 1024 && raised[channel_decay ? 1 : 0] < smem) {                                                \
            e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                       \
            if (e != cudaSuccess) return (int)e;                                                                       \
            raised[channel_decay ? 1 : 0] = smem;                                                                      \
        }                                                                                                              \
        e = launch_pdl(k, grid, dim3(DR_THREADS), smem, stream, qk, v, g, beta, state, slots, cu_seqlens, out, out_stride, H, \
                       G, Dp, V, Vp);                                                                                  \
    } while (0)
    ZLM_DR_SHAPES(ZLM_DR_SCAN)
#undef ZLM_DR_SCAN
    return e == cudaSuccess ? launch_status() : (int)e;
}

template <typename T>
static int dr_decode_launch(const DrIn<T>& in, int channel_decay, int n_seqs, float* state, const float* norm_w, float eps,
                            const void* gate, long gate_stride, int gate_kind, void* out, long out_stride,
                            cudaStream_t stream) {
    int L, NI;
    if (!dr_shape(in.Dp, L, NI) || n_seqs > 65535) return ZLM_ERR_UNSUPPORTED;
    int threads = (in.V * L + 31) / 32 * 32;
    threads = threads < 64 ? 64 : (threads > 1024 ? 1024 : threads);
    if (NI > 4 && threads > 512) threads = 512;
    const size_t smem = ((size_t)3 * 4 * L * NI + 2 * in.V) * sizeof(float);
    if (smem > 48 * 1024) return ZLM_ERR_UNSUPPORTED;
    dim3 grid(in.H, n_seqs);
    cudaError_t e = cudaSuccess;
#define ZLM_DR_DEC(LL, NN)                                                                                             \
    do {                                                                                                               \
        auto* k = channel_decay ? dr_decode_kernel<T, LL, NN, true> : dr_decode_kernel<T, LL, NN, false>;              \
        e = launch_pdl(k, grid, dim3(threads), smem, stream, in, state, norm_w, eps, (const T*)gate, gate_stride, gate_kind, \
                       (T*)out, out_stride);                                                                           \
    } while (0)
    ZLM_DR_SHAPES(ZLM_DR_DEC)
#undef ZLM_DR_DEC
    return e == cudaSuccess ? launch_status() : (int)e;
}

// One token a sequence (row b of proj belongs to sequence b).  gate: rows of H V numbers of proj's type, or null;
// gate_kind 1 sigmoid, 2 silu; norm_w: float [V]; out: rows of H V numbers of proj's type.
ZLM_EXPORT int zlm_delta_decode(const void* proj, int dtype, long proj_stride, const float* taps, float* ring, int H, int G,
                                int D, int V, int K, const float* a, long a_stride, int channel_decay, const float* b,
                                long b_stride, const float* rate, const float* dt_bias, const int* slots,
                                const int* past_lens, int n_seqs, float* state, const float* norm_w, float eps,
                                const void* gate, long gate_stride, int gate_kind, void* out, long out_stride,
                                cudaStream_t stream) {
    if (n_seqs <= 0) return 0;
    if (dtype == ZLM_F32) {
        DrIn<float> in;
        const int s = dr_fill<float>(in, proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, b, b_stride, rate, dt_bias,
                                     slots, past_lens, nullptr);
        return s ? s : dr_decode_launch<float>(in, channel_decay, n_seqs, state, norm_w, eps, gate, gate_stride, gate_kind, out,
                                               out_stride, stream);
    }
    if (dtype == ZLM_BF16) {
        DrIn<__nv_bfloat16> in;
        const int s = dr_fill<__nv_bfloat16>(in, proj, proj_stride, taps, ring, H, G, D, V, K, a, a_stride, b, b_stride, rate,
                                             dt_bias, slots, past_lens, nullptr);
        return s ? s : dr_decode_launch<__nv_bfloat16>(in, channel_decay, n_seqs, state, norm_w, eps, gate, gate_stride,
                                                       gate_kind, out, out_stride, stream);
    }
    return ZLM_ERR_UNSUPPORTED;
}
