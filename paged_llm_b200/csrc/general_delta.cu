// The generalized delta rule: a matrix state per head with a decay and a removal rate per key channel.
//
//     S <- diag(w) S - (a u) (u^T S) + k v^T,   o = S^T r          u = k / sqrt(sum k^2 + unit_eps), both terms from the old S
//     w = exp(decay_scale * sigmoid(z + w0)),   a = sigmoid(removal + removal bias)
//
// and the causal convolution per channel that is added to a mixer's input.  Everything is float32 whatever the
// activations' type is; the state of a request lives in a slot of [slots, state_stride] floats, a head's state column by
// column ([H][d][d], column j the d numbers S[:, j]).  Few tokens per request run the recurrence token by token, prompt portions
// in short chunks whose tokens are worked on together; every sum has a fixed order that does not depend on the batch.
#include "common.cuh"

namespace {

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }

// ------------------------------------------------------------------ h + conv(h)
// out[t, c] = h[t, c] + sum_j w[c, j] h[t - taps + 1 + j, c], inputs in front of the step from the state's first
// (taps-1) * C floats ([taps-1][C]), which are then replaced by the step's last inputs.  grid: (requests, channel blocks,
// token chunks of RC_TOK); 32 lanes of VEC channels x token lanes.  The block of chunk 0 alone reads the old inputs and
// writes the new ones, after a barrier.
constexpr int RC_TOK = 32;

template <typename T, int VEC>
__device__ __forceinline__ void rc_load(const T* p, float (&v)[VEC]) {
    if (VEC == 4) {
        if (sizeof(T) == 4) {
            const float4 a = *reinterpret_cast<const float4*>(p);
            v[0] = a.x, v[VEC > 1 ? 1 : 0] = a.y, v[VEC > 2 ? 2 : 0] = a.z, v[VEC > 3 ? 3 : 0] = a.w;
        } else {
            const uint2 raw = *reinterpret_cast<const uint2*>(p);
            const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
            v[0] = __low2float(a), v[VEC > 1 ? 1 : 0] = __high2float(a), v[VEC > 2 ? 2 : 0] = __low2float(b), v[VEC > 3 ? 3 : 0] = __high2float(b);
        }
    } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) v[i] = to_float(p[i]);
    }
}
template <typename T, int VEC>
__device__ __forceinline__ void rc_store(T* p, const float (&v)[VEC]) {
#pragma unroll
    for (int i = 0; i < VEC; ++i) p[i] = from_float<T>(v[i]);
}
template <>
__device__ __forceinline__ void rc_store<float, 4>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <>
__device__ __forceinline__ void rc_store<__nv_bfloat16, 4>(__nv_bfloat16* p, const float (&v)[4]) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&lo);
    raw.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(p) = raw;
}

// cw: [taps][C] (a tap's weights of all channels side by side)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) residual_conv_kernel(const T* __restrict__ h, int C, const float* __restrict__ cw, int taps,
                                                            float* __restrict__ state, long long state_stride,
                                                            const int* __restrict__ cu_q, const int* __restrict__ slots,
                                                            T* __restrict__ out) {
    pdl_launch_dependents();
    const int s = blockIdx.x;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    const int t_lo = blockIdx.z * RC_TOK, t_hi = min(nq, t_lo + RC_TOK);
    const int c = (blockIdx.y * 32 + threadIdx.x) * VEC;
    pdl_wait();
    const int hist = taps - 1;
    if ((slot < 0 && hist > 0) || t_lo >= nq) return;
    const bool ok = c < C;
    float* st = hist > 0 ? state + (size_t)slot * state_stride + (ok ? c : 0) : nullptr;
    const T* col = h + (size_t)q0 * C + (ok ? c : 0);
    auto input = [&](int src, float (&v)[VEC]) {
        if (src >= 0) rc_load<T, VEC>(col + (size_t)src * C, v);
        else rc_load<float, VEC>(st + (size_t)(hist + src) * C, v);
    };
    if (ok) {
        for (int t = t_lo + threadIdx.y; t < t_hi; t += blockDim.y) {
            float acc[VEC], self[VEC];
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc[i] = 0.f;
            for (int j = 0; j < taps; ++j) {
                float w[VEC];
                rc_load<float, VEC>(cw + (size_t)j * C + c, w);
                input(t - hist + j, self);
#pragma unroll
                for (int i = 0; i < VEC; ++i) acc[i] = fmaf(w[i], self[i], acc[i]);
            }
#pragma unroll
            for (int i = 0; i < VEC; ++i) acc[i] += self[i];          // (the last tap's input is the token itself)
            rc_store<T, VEC>(out + (size_t)(q0 + t) * C + c, acc);
        }
    }
    if (blockIdx.z != 0 || hist == 0) return;
    __syncthreads();                                                  // every read of the old inputs is done
    if (ok && threadIdx.y == 0) {
        // the last taps-1 inputs of [old inputs ; this step's]: in place from the front, since entry j reads old entry
        // j + nq > j or a new input
        for (int j = 0; j < hist; ++j) {
            float v[VEC];
            input(nq + j - hist, v);
            rc_store<float, VEC>(st + (size_t)j * C, v);
        }
    }
}

// ------------------------------------------------------------------ the generalized delta rule
// Columns of a row of the input projection (row stride ld): [r: C | k: C | v: C | g: C | removal: C | decay: rank], C = H * d.
struct GdIn {
    const void* proj;
    int ld;
    const float *w0, *a_bias;   // [C]
    int H, d;
    float decay_scale, unit_eps;
};

// Per token and head, what does not depend on the state: w, u, a u, k, r w, v and the numbers r . (a u) and r . k.  A warp
// computes one (token, head); `lane` takes channels lane, lane + 32, ...; z: the head's d decay inputs in front of their bias.
template <typename T>
__device__ __forceinline__ void gd_prepare(const GdIn& in, long long t, int h, int lane, const float* z, float* w, float* u, float* au,
                                           float* k, float* rw, float* v, float* scal) {
    const int d = in.d, C = in.H * d, c0 = h * d;
    const T* row = (const T*)in.proj + (size_t)t * in.ld + c0;
    float sq = 0.f;
    for (int i = lane; i < d; i += 32) {
        const float kv = to_float(row[C + i]);
        sq = fmaf(kv, kv, sq);
    }
    const float f = 1.0f / sqrtf(warp_sum(sq) + in.unit_eps);
    float rau = 0.f, rk = 0.f;
    for (int i = lane; i < d; i += 32) {
        const float rv = to_float(row[i]), kv = to_float(row[C + i]);
        const float a = sigmoid_f(to_float(row[4 * C + i]) + __ldg(in.a_bias + c0 + i));
        const float wv = expf(in.decay_scale * sigmoid_f(z[i] + __ldg(in.w0 + c0 + i)));
        const float uv = kv * f, auv = a * uv;
        w[i] = wv, u[i] = uv, au[i] = auv, k[i] = kv, rw[i] = rv * wv, v[i] = to_float(row[2 * C + i]);
        rau = fmaf(rv, auv, rau);
        rk = fmaf(rv, kv, rk);
    }
    rau = warp_sum(rau);
    rk = warp_sum(rk);
    if (lane == 0) scal[0] = rau, scal[1] = rk;
}

// ------------------------------------------------------------------ few tokens per request (decoding)
// A block per (request, head) does the whole mixer between its two projections: the decay's low rank
// (tanh, product), gates and unit norm, the recurrence, the norm of the head's output and the output gate.  The head's state
// travels to shared memory while the rest is prepared.  Eight lanes share a column of it, lane l holding the key channels
// 4 l + 32 m + (0..3), m < NPER / 4.  Per column and token, with the dots summed over the lanes by one butterfly:
//     c = u . S_j,  e = (r w) . S_j,  S_j <- w S_j - (a u) c + k v_j,  o_j = e - (r . a u) c + (r . k) v_j
struct GdTail {
    const void* w_decay;        // [C][rank]
    int rank;                   // a multiple of 8, at most GD_MAX_RANK
    const float* norm_w;        // [C]
    float eps;
};
constexpr int GD_MAX_RANK = 256, GS_TOK = 4, GS_THREADS = 256, GS_LANES = 8;

__device__ __forceinline__ void gs_load8(const float* p, float (&v)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
__device__ __forceinline__ void gs_load8(const __nv_bfloat16* p, float (&v)[8]) {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[2 * i] = __low2float(h[i]), v[2 * i + 1] = __high2float(h[i]);
}

__device__ __forceinline__ void gd_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

__host__ __device__ constexpr int gs_smem(int DP) { return (DP * DP + GS_TOK * (6 * DP + 4) + GS_TOK * DP + GS_TOK * GD_MAX_RANK) * (int)sizeof(float); }

template <typename T, int NPER>
__global__ void __launch_bounds__(GS_THREADS) gd_step_kernel(GdIn in, GdTail tail, float* __restrict__ state, long long state_stride,
                                                             const int* __restrict__ cu_q, const int* __restrict__ slots,
                                                             T* __restrict__ out, int vec) {
    constexpr int DP = NPER * GS_LANES, ROW = 6 * DP + 4;
    extern __shared__ __align__(16) float gs_raw[];
    float* Ss = gs_raw;                                 // [DP columns][DP]: the head's state
    float* rows = Ss + DP * DP;                         // [GS_TOK][ROW]
    float* zs = rows + GS_TOK * ROW;                    // [GS_TOK][DP]: the decay's inputs, then the head's outputs
    float* th = zs + GS_TOK * DP;                       // [GS_TOK][GD_MAX_RANK]
    pdl_launch_dependents();
    const int s = blockIdx.x / in.H, h = blockIdx.x - s * in.H, d = in.d, C = in.H * d, c0 = h * d;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    const int tid = threadIdx.x, lane = tid % GS_LANES, col = tid / GS_LANES, wlane = tid & 31, warp = tid >> 5;
    if (slot < 0 || nq <= 0) {
        pdl_wait();
        return;
    }
    // (the state was left by the step before, not by the kernel in front)
    float* sp = state + (size_t)slot * state_stride + (size_t)h * d * d;
    if (vec) {
        for (int e = tid; e < d * (DP / 4); e += GS_THREADS) {
            const int j = e / (DP / 4), ch = (e - j * (DP / 4)) * 4;
            if (ch < d) gd_cp16(Ss + j * DP + ch, sp + (size_t)j * d + ch);
            else *reinterpret_cast<float4*>(Ss + j * DP + ch) = make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
        for (int e = tid; e < d * DP; e += GS_THREADS) {
            const int j = e / DP, ch = e - j * DP;
            Ss[e] = ch < d ? sp[(size_t)j * d + ch] : 0.f;
        }
    }
    asm volatile("cp.async.commit_group;\n" ::);
    pdl_wait();
    if (d < DP)
        for (int e = tid; e < GS_TOK * ROW; e += GS_THREADS) rows[e] = 0.f;          // channels that pad a row stay zero
    const T* proj = (const T*)in.proj;
    for (int t0 = 0; t0 < nq; t0 += GS_TOK) {
        const int nt = min(GS_TOK, nq - t0);
        const bool last = t0 + GS_TOK >= nq;
        for (int e = tid; e < nt * tail.rank; e += GS_THREADS) {
            const int tt = e / tail.rank, r = e - tt * tail.rank;
            // (rounded as the activations of a product are)
            th[tt * GD_MAX_RANK + r] = to_float(from_float<T>(tanhf(to_float(proj[(size_t)(q0 + t0 + tt) * in.ld + 5 * C + r]))));
        }
        __syncthreads();
        for (int e = tid; e < nt * d; e += GS_THREADS) {
            const int tt = e / d, i = e - tt * d;
            const T* w2 = (const T*)tail.w_decay + (size_t)(c0 + i) * tail.rank;
            float acc = 0.f;
#pragma unroll 4
            for (int r = 0; r < tail.rank; r += 8) {
                float w8[8];
                gs_load8(w2 + r, w8);
#pragma unroll
                for (int q = 0; q < 8; ++q) acc = fmaf(th[tt * GD_MAX_RANK + r + q], w8[q], acc);
            }
            zs[tt * DP + i] = acc;
        }
        __syncthreads();
        if (warp < nt) {
            float* o = rows + warp * ROW;
            gd_prepare<T>(in, q0 + t0 + warp, h, wlane, zs + warp * DP, o, o + DP, o + 2 * DP, o + 3 * DP, o + 4 * DP, o + 5 * DP, o + 6 * DP);
        }
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();
#pragma unroll 2
        for (int j = col; j < DP; j += GS_THREADS / GS_LANES) {       // (uniform per warp: a multiple of its four columns)
            float S[NPER];
            const int jr = j < d ? j : 0;
#pragma unroll
            for (int m = 0; m < NPER / 4; ++m) {
                const float4 v = *reinterpret_cast<const float4*>(Ss + jr * DP + m * 32 + lane * 4);
                S[4 * m] = v.x, S[4 * m + 1] = v.y, S[4 * m + 2] = v.z, S[4 * m + 3] = v.w;
            }
            for (int tt = 0; tt < nt; ++tt) {
                const float* row = rows + tt * ROW;
                const float rau = row[6 * DP], rk = row[6 * DP + 1], v = row[5 * DP + jr];
                float c4[4] = {0.f, 0.f, 0.f, 0.f}, e4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int m = 0; m < NPER / 4; ++m) {
                    const float4 u4 = *reinterpret_cast<const float4*>(row + DP + m * 32 + lane * 4);
                    const float4 q4 = *reinterpret_cast<const float4*>(row + 4 * DP + m * 32 + lane * 4);
                    c4[0] = fmaf(S[4 * m], u4.x, c4[0]), c4[1] = fmaf(S[4 * m + 1], u4.y, c4[1]);
                    c4[2] = fmaf(S[4 * m + 2], u4.z, c4[2]), c4[3] = fmaf(S[4 * m + 3], u4.w, c4[3]);
                    e4[0] = fmaf(S[4 * m], q4.x, e4[0]), e4[1] = fmaf(S[4 * m + 1], q4.y, e4[1]);
                    e4[2] = fmaf(S[4 * m + 2], q4.z, e4[2]), e4[3] = fmaf(S[4 * m + 3], q4.w, e4[3]);
                }
                float c = (c4[0] + c4[1]) + (c4[2] + c4[3]);
                const float e = (e4[0] + e4[1]) + (e4[2] + e4[3]);
                // after the first step the lower half of a column's lanes carries the partial sums of c, the upper half
                // those of e; c then goes to every lane from the column's first
                const bool upper = lane >= GS_LANES / 2;
                float x = upper ? e : c;
                x += __shfl_xor_sync(0xffffffffu, upper ? c : e, GS_LANES / 2);
#pragma unroll
                for (int o = GS_LANES / 4; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
                c = __shfl_sync(0xffffffffu, x, wlane & ~(GS_LANES - 1));
#pragma unroll
                for (int m = 0; m < NPER / 4; ++m) {
                    const float4 w4 = *reinterpret_cast<const float4*>(row + m * 32 + lane * 4);
                    const float4 a4 = *reinterpret_cast<const float4*>(row + 2 * DP + m * 32 + lane * 4);
                    const float4 k4 = *reinterpret_cast<const float4*>(row + 3 * DP + m * 32 + lane * 4);
                    S[4 * m] = fmaf(-a4.x, c, fmaf(w4.x, S[4 * m], k4.x * v));
                    S[4 * m + 1] = fmaf(-a4.y, c, fmaf(w4.y, S[4 * m + 1], k4.y * v));
                    S[4 * m + 2] = fmaf(-a4.z, c, fmaf(w4.z, S[4 * m + 2], k4.z * v));
                    S[4 * m + 3] = fmaf(-a4.w, c, fmaf(w4.w, S[4 * m + 3], k4.w * v));
                }
                if (j < d && lane == GS_LANES / 2) zs[tt * DP + j] = fmaf(rk, v, fmaf(-rau, c, x));
            }
            if (j < d) {
#pragma unroll
                for (int m = 0; m < NPER / 4; ++m) {
                    const int ch = m * 32 + lane * 4;
                    const float4 v = make_float4(S[4 * m], S[4 * m + 1], S[4 * m + 2], S[4 * m + 3]);
                    if (!last) *reinterpret_cast<float4*>(Ss + j * DP + ch) = v;
                    else if (vec) {
                        if (ch < d) *reinterpret_cast<float4*>(sp + (size_t)j * d + ch) = v;
                    } else {
#pragma unroll
                        for (int q = 0; q < 4; ++q)
                            if (ch + q < d) sp[(size_t)j * d + ch + q] = S[4 * m + q];
                    }
                }
            }
        }
        __syncthreads();
        if (warp < nt) {
            const float* o = zs + warp * DP;
            float sq = 0.f;
            for (int i = wlane; i < d; i += 32) sq = fmaf(o[i], o[i], sq);
            const float f = 1.0f / sqrtf(warp_sum(sq) / (float)d + tail.eps);
            const T* g = proj + (size_t)(q0 + t0 + warp) * in.ld + 3 * C + c0;
            T* dst = out + (size_t)(q0 + t0 + warp) * C + c0;
            for (int i = wlane; i < d; i += 32) dst[i] = from_float<T>(o[i] * f * __ldg(tail.norm_w + c0 + i) * sigmoid_f(to_float(g[i])));
        }
        __syncthreads();
    }
}

template <typename T, int NPER>
int launch_gd_step_as(const GdIn& in, const GdTail& tail, float* state, long long state_stride, const int* cu_q, const int* slots, int num_seqs,
                      void* out, cudaStream_t stream) {
    const int vec = in.d % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    constexpr int smem = gs_smem(NPER * GS_LANES);
    static bool opted = false;
    if (!opted) {
        PL_CUDA(cudaFuncSetAttribute(gd_step_kernel<T, NPER>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        opted = true;
    }
    PL_CUDA(launch_pdl(gd_step_kernel<T, NPER>, dim3((unsigned)num_seqs * in.H), dim3(GS_THREADS), (size_t)smem, stream, in, tail, state,
                       state_stride, cu_q, slots, (T*)out, vec));
    return 0;
}

template <typename T>
int launch_gd_step(const GdIn& in, const GdTail& tail, float* state, long long state_stride, const int* cu_q, const int* slots, int num_seqs,
                   void* out, cudaStream_t stream) {
    if (in.d <= 32) return launch_gd_step_as<T, 4>(in, tail, state, state_stride, cu_q, slots, num_seqs, out, stream);
    if (in.d <= 64) return launch_gd_step_as<T, 8>(in, tail, state, state_stride, cu_q, slots, num_seqs, out, stream);
    return launch_gd_step_as<T, 16>(in, tail, state, state_stride, cu_q, slots, num_seqs, out, stream);
}

// ------------------------------------------------------------------ prompt portions: chunks of GC tokens
// With P_t the product of the decays from the chunk's start through token t (per channel), and
//     x_t = P_(t-1) u_t,   b_t = (a u)_t / P_t,   k~_t = k_t / P_t,   y_t = P_t r_t,
// the recurrence inside a chunk that starts from the state S is, with c_t = u_t^T S_(t-1) (a row over the columns),
//     c_t = x_t^T S + sum_(s<t)  [ (x_t . k~_s) v_s - (x_t . b_s) c_s ]
//     o_t = y_t^T S + sum_(s<=t) [ (y_t . k~_s) v_s - (y_t . b_s) c_s ]
//     S'  = diag(P_end) (S + sum_s [ k~_s v_s^T - b_s c_s^T ])
// Solving the triangular system for c leaves c = X S + G V and o = Y S + H V with matrices that do not depend on the state.
// The first kernel forms them for all chunks at once; the second walks a request's chunks in order, and per chunk multiplies
// [X | G; Y | H] by the state over the chunk's values, then adds the chunk to the state.  A decay is at least exp(decay_scale)
// and a chunk is short, so 1 / P stays far inside float32's range.
// The chunks of request s are numbered from cu_q[s] / GC + s; the numbers of different requests do not meet.
constexpr int GC = 16, GC_THREADS = 256, GC_COLS = 16;

// Floats of a (chunk, head): [DP + GC][2 GC] the matrix above, transposed; [2 GC][DP] what is added to the state per value and
// per c; [DP] P_end; [GC][DP] the values.
__host__ __device__ constexpr size_t gc_floats(int DP) { return (size_t)(DP + GC) * 2 * GC + 2 * GC * DP + DP + GC * DP; }
__host__ __device__ constexpr int gc_prepare_smem(int DP) { return (4 * GC * (DP + 4) + 4 * GC * GC + GC) * (int)sizeof(float); }

template <typename T, int DP>
__global__ void __launch_bounds__(GC_THREADS) gd_chunk_prepare_kernel(GdIn in, const float* __restrict__ z, const int* __restrict__ cu_q,
                                                                      const int* __restrict__ slots, int num_seqs, float* __restrict__ buf) {
    constexpr int LD = DP + 4;                          // rows 4 floats longer: 16-byte reads of eight rows meet no bank twice
    extern __shared__ __align__(16) float gc_smem[];
    float *xs = gc_smem, *bs = xs + GC * LD, *ks = bs + GC * LD, *ys = ks + GC * LD;      // first w, a; then x, b, k~, y
    float* gram = ys + GC * LD;                         // [x . k~ | x . b | y . k~ | y . b][GC][GC]
    float* unit = gram + 4 * GC * GC;                   // [GC]
    const int chunk = blockIdx.x, h = blockIdx.y, d = in.d, C = in.H * d, c0 = h * d;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    // the request this chunk belongs to: the last one whose first chunk number is not above it
    int lo = 0, hi = num_seqs - 1;
    while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (cu_q[mid] / GC + mid <= chunk) lo = mid;
        else hi = mid - 1;
    }
    const int s = lo, q0 = cu_q[s], nq = cu_q[s + 1] - q0, t0 = (chunk - q0 / GC - s) * GC;
    if (t0 < 0 || t0 >= nq || slots[s] < 0) return;
    const int nt = min(GC, nq - t0);
    const T* row0 = (const T*)in.proj + (size_t)(q0 + t0) * in.ld + c0;
    const float* z0 = z + (size_t)(q0 + t0) * C + c0;
    for (int t = warp; t < nt; t += GC_THREADS / 32) {
        float sq = 0.f;
        for (int i = lane; i < d; i += 32) {
            const float kv = to_float(row0[(size_t)t * in.ld + C + i]);
            sq = fmaf(kv, kv, sq);
        }
        sq = warp_sum(sq);
        if (lane == 0) unit[t] = 1.0f / sqrtf(sq + in.unit_eps);
    }
    for (int e = tid; e < GC * DP; e += GC_THREADS) {
        const int t = e / DP, i = e - t * DP;
        float w = 1.f, a = 0.f;
        if (t < nt && i < d) {
            w = expf(in.decay_scale * sigmoid_f(z0[(size_t)t * C + i] + __ldg(in.w0 + c0 + i)));
            a = sigmoid_f(to_float(row0[(size_t)t * in.ld + 4 * C + i]) + __ldg(in.a_bias + c0 + i));
        }
        xs[t * LD + i] = w;
        bs[t * LD + i] = a;
    }
    __syncthreads();
    float* M = buf + ((size_t)chunk * in.H + h) * gc_floats(DP);
    float* W = M + (size_t)(DP + GC) * 2 * GC;
    float* Pend = W + 2 * GC * DP;
    float* V = Pend + DP;
    for (int i = tid; i < DP; i += GC_THREADS) {
        float P = 1.f, invs[GC], kk[GC], ab[GC];
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            float r = 0.f, k = 0.f, v = 0.f, f = 0.f;
            if (t < nt && i < d) {
                const T* row = row0 + (size_t)t * in.ld + i;
                r = to_float(row[0]), k = to_float(row[C]), v = to_float(row[2 * C]), f = unit[t];
            }
            const float u = k * f, au = bs[t * LD + i] * u, w = xs[t * LD + i];
            xs[t * LD + i] = P * u;
            P *= w;
            const float inv = 1.0f / P;
            invs[t] = inv, kk[t] = k * inv, ab[t] = au * inv;
            bs[t * LD + i] = ab[t];
            ks[t * LD + i] = kk[t];
            ys[t * LD + i] = P * r;
            V[t * DP + i] = v;
        }
        Pend[i] = P;
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            W[t * DP + i] = kk[t] * P;
            W[(GC + t) * DP + i] = -ab[t] * P;
        }
    }
    __syncthreads();
    {
        // a thread per pair (t, s): four dots
        const int t = tid / GC, q = tid - t * GC;
        float xk = 0.f, xb = 0.f, yk = 0.f, yb = 0.f;
        for (int i = 0; i < DP; i += 4) {
            const float4 x = *reinterpret_cast<const float4*>(xs + t * LD + i), y = *reinterpret_cast<const float4*>(ys + t * LD + i);
            const float4 k = *reinterpret_cast<const float4*>(ks + q * LD + i), b = *reinterpret_cast<const float4*>(bs + q * LD + i);
            xk = fmaf(x.x, k.x, fmaf(x.y, k.y, fmaf(x.z, k.z, fmaf(x.w, k.w, xk))));
            xb = fmaf(x.x, b.x, fmaf(x.y, b.y, fmaf(x.z, b.z, fmaf(x.w, b.w, xb))));
            yk = fmaf(y.x, k.x, fmaf(y.y, k.y, fmaf(y.z, k.z, fmaf(y.w, k.w, yk))));
            yb = fmaf(y.x, b.x, fmaf(y.y, b.y, fmaf(y.z, b.z, fmaf(y.w, b.w, yb))));
        }
        gram[t * GC + q] = q < t ? xk : 0.f;
        gram[GC * GC + t * GC + q] = q < t ? xb : 0.f;
        gram[2 * GC * GC + t * GC + q] = q <= t ? yk : 0.f;
        gram[3 * GC * GC + t * GC + q] = q <= t ? yb : 0.f;
    }
    __syncthreads();
    // forward substitution, a thread per column of [X | G], then the same column of [Y | H]
    for (int c = tid; c < DP + GC; c += GC_THREADS) {
        float x[GC];
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            float acc = c < DP ? xs[t * LD + c] : gram[t * GC + c - DP];
#pragma unroll
            for (int q = 0; q < t; ++q) acc = fmaf(-gram[GC * GC + t * GC + q], x[q], acc);
            x[t] = acc;
        }
        float* m = M + (size_t)c * 2 * GC;
#pragma unroll
        for (int t = 0; t < GC; t += 4) *reinterpret_cast<float4*>(m + t) = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
        float o[4];
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            float acc = c < DP ? ys[t * LD + c] : gram[2 * GC * GC + t * GC + c - DP];
#pragma unroll
            for (int q = 0; q <= t; ++q) acc = fmaf(-gram[3 * GC * GC + t * GC + q], x[q], acc);
            o[t & 3] = acc;
            if ((t & 3) == 3) *reinterpret_cast<float4*>(m + GC + t - 3) = make_float4(o[0], o[1], o[2], o[3]);
        }
    }
}

// Shared floats of the second kernel: two stages of [matrix | additions | P_end | a block of the values], the state's block
// of columns, c, and the partial sums of eight warps.
__host__ __device__ constexpr int gc_stage_floats(int DP) { return (DP + GC) * 2 * GC + 2 * GC * DP + DP + GC * GC_COLS; }
__host__ __device__ constexpr int gc_scan_smem(int DP) {
    return (2 * gc_stage_floats(DP) + DP * GC_COLS + GC * GC_COLS + 8 * 2 * GC * GC_COLS) * (int)sizeof(float);
}

// grid: (requests, heads, blocks of 16 columns); 256 threads.  Per chunk: the 2 GC x 16 product over the DP + GC rows of state
// and values, cut between the eight warps (tiles of 4 x 4 per thread) and summed in a fixed order; then the state's update.
template <int DP>
__global__ void __launch_bounds__(GC_THREADS) gd_chunk_scan_kernel(int H, int d, const float* __restrict__ buf, float* __restrict__ state,
                                                                   long long state_stride, const int* __restrict__ cu_q,
                                                                   const int* __restrict__ slots, float* __restrict__ out) {
    constexpr int STAGE = gc_stage_floats(DP), KW = (DP + GC) / 8, MF = (DP + GC) * 2 * GC + 2 * GC * DP + DP;
    static_assert((DP + GC) % 8 == 0 && MF % 4 == 0, "");
    extern __shared__ __align__(16) float gc_smem_raw[];
    float* Ss = gc_smem_raw + 2 * STAGE;                // [DP][16]
    float* Cs = Ss + DP * GC_COLS;                      // [GC][16]
    float* part = Cs + GC * GC_COLS;                    // [8][2 GC][16]
    const int s = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * GC_COLS;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    if (slot < 0 || nq <= 0) return;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    float* sp = state + (size_t)slot * state_stride + (size_t)h * d * d;
    const size_t per = gc_floats(DP);
    const float* src0 = buf + ((size_t)(q0 / GC + s) * H + h) * per;
    const int chunks = (nq + GC - 1) / GC;
    auto stage = [&](int c, int b) {
        float* dst = gc_smem_raw + b * STAGE;
        const float* src = src0 + (size_t)c * H * per;
        for (int e = tid; e < MF / 4; e += GC_THREADS) gd_cp16(dst + e * 4, src + e * 4);
        const float* v = src + MF + j0;                 // the values' columns j0 .. j0 + 15 (DP is a multiple of 16)
        if (tid < GC * GC_COLS / 4) gd_cp16(dst + MF + tid * 4, v + (tid >> 2) * DP + (tid & 3) * 4);
        asm volatile("cp.async.commit_group;\n" ::);
    };
    stage(0, 0);
    for (int e = tid; e < GC_COLS * DP; e += GC_THREADS) {
        const int j = e / DP, k = e - j * DP;
        Ss[k * GC_COLS + j] = j0 + j < d && k < d ? sp[(size_t)(j0 + j) * d + k] : 0.f;
    }
    const int rt = (lane >> 2) * 4, ct = (lane & 3) * 4;             // the product's tile of this thread
    constexpr int R = DP >= 64 ? DP / 64 : 1;                        // rows of the state's tile
    const int sr = (tid >> 2) * R, sc = (tid & 3) * 4;
    const bool owns = sr < DP;
    for (int c = 0; c < chunks; ++c) {
        const int b = c & 1, nt = min(GC, nq - c * GC);
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();
        if (c + 1 < chunks) stage(c + 1, b ^ 1);
        const float* M = gc_smem_raw + b * STAGE;
        const float* W = M + (DP + GC) * 2 * GC;
        const float* Pend = W + 2 * GC * DP;
        const float* V = Pend + DP;
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 6
        for (int kk = 0; kk < KW; ++kk) {
            const int k = warp * KW + kk;
            const float4 m = *reinterpret_cast<const float4*>(M + k * 2 * GC + rt);
            const float4 x = *reinterpret_cast<const float4*>((k < DP ? Ss + k * GC_COLS : V + (k - DP) * GC_COLS) + ct);
            const float mm[4] = {m.x, m.y, m.z, m.w}, xx[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(mm[i], xx[j], acc[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
            *reinterpret_cast<float4*>(part + (warp * 2 * GC + rt + i) * GC_COLS + ct) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        // what does not wait for c: the decayed state and the values' part
        float st[R][4];
        if (owns) {
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float p = Pend[sr + r];
                const float4 x = *reinterpret_cast<const float4*>(Ss + (sr + r) * GC_COLS + sc);
                st[r][0] = p * x.x, st[r][1] = p * x.y, st[r][2] = p * x.z, st[r][3] = p * x.w;
            }
#pragma unroll 4
            for (int q = 0; q < GC; ++q) {
                const float4 x = *reinterpret_cast<const float4*>(V + q * GC_COLS + sc);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float w = W[q * DP + sr + r];
                    st[r][0] = fmaf(w, x.x, st[r][0]), st[r][1] = fmaf(w, x.y, st[r][1]);
                    st[r][2] = fmaf(w, x.z, st[r][2]), st[r][3] = fmaf(w, x.w, st[r][3]);
                }
            }
        }
        __syncthreads();
        {
            const int row = tid >> 3, col = (tid & 7) * 2;
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float2 x = *reinterpret_cast<const float2*>(part + (w * 2 * GC + row) * GC_COLS + col);
                a0 += x.x, a1 += x.y;
            }
            if (row < GC) {
                *reinterpret_cast<float2*>(Cs + row * GC_COLS + col) = make_float2(a0, a1);
            } else if (row - GC < nt) {
                float* o = out + ((size_t)(q0 + c * GC + row - GC) * H + h) * d + j0 + col;
                if (j0 + col < d) o[0] = a0;
                if (j0 + col + 1 < d) o[1] = a1;
            }
        }
        __syncthreads();
        if (owns) {
#pragma unroll 4
            for (int q = 0; q < GC; ++q) {
                const float4 x = *reinterpret_cast<const float4*>(Cs + q * GC_COLS + sc);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    const float w = W[(GC + q) * DP + sr + r];
                    st[r][0] = fmaf(w, x.x, st[r][0]), st[r][1] = fmaf(w, x.y, st[r][1]);
                    st[r][2] = fmaf(w, x.z, st[r][2]), st[r][3] = fmaf(w, x.w, st[r][3]);
                }
            }
#pragma unroll
            for (int r = 0; r < R; ++r)
                *reinterpret_cast<float4*>(Ss + (sr + r) * GC_COLS + sc) = make_float4(st[r][0], st[r][1], st[r][2], st[r][3]);
        }
    }
    __syncthreads();
    for (int e = tid; e < GC_COLS * DP; e += GC_THREADS) {
        const int j = e / DP, k = e - j * DP;
        if (j0 + j < d && k < d) sp[(size_t)(j0 + j) * d + k] = Ss[k * GC_COLS + j];
    }
}

template <typename T, int DP>
int launch_gd_chunks(const GdIn& in, const float* z, float* buf, int slots_of_chunks, float* state, long long state_stride, const int* cu_q,
                     const int* slots, int num_seqs, float* out, cudaStream_t stream) {
    static bool opted = false;
    if (!opted) {
        PL_CUDA(cudaFuncSetAttribute(gd_chunk_prepare_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, gc_prepare_smem(DP)));
        PL_CUDA(cudaFuncSetAttribute(gd_chunk_scan_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, gc_scan_smem(DP)));
        opted = true;
    }
    PL_REQUIRE(in.H <= 65535, "general_delta: %d heads", in.H);
    gd_chunk_prepare_kernel<T, DP><<<dim3(slots_of_chunks, in.H), GC_THREADS, gc_prepare_smem(DP), stream>>>(in, z, cu_q, slots, num_seqs, buf);
    PL_LAUNCHED("general_delta_chunk_prepare");
    gd_chunk_scan_kernel<DP><<<dim3(num_seqs, in.H, (in.d + GC_COLS - 1) / GC_COLS), GC_THREADS, gc_scan_smem(DP), stream>>>(
        in.H, in.d, buf, state, state_stride, cu_q, slots, out);
    PL_LAUNCHED("general_delta_chunk_scan");
    return 0;
}

}  // namespace

// `max_tokens`: no request of the step brings more.  h, out: [T, C] in `dtype`; cw: [taps][C] float32.
PL_EXPORT int pl_residual_conv(const void* h, int dtype, int C, const float* cw, int taps, float* state, long long state_stride,
                               const int* cu_q, const int* slots, int num_seqs, int max_tokens, void* out, cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    PL_REQUIRE(C > 0 && taps >= 1 && taps <= RC_TOK && max_tokens >= 1, "residual_conv: bad sizes C=%d taps=%d (at most %d)", C, taps, RC_TOK);
    PL_REQUIRE(taps == 1 || (state != nullptr && state_stride >= (long long)(taps - 1) * C), "residual_conv: no room for the last inputs");
    const bool vec = C % 4 == 0 && state_stride % 4 == 0 && (((uintptr_t)h | (uintptr_t)out | (uintptr_t)cw | (uintptr_t)state) & 15) == 0;
    const int per = vec ? 128 : 32;
    const dim3 grid(num_seqs, (C + per - 1) / per, (max_tokens + RC_TOK - 1) / RC_TOK), block(32, max_tokens == 1 ? 1 : 8);
    PL_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "residual_conv: %d tokens of %d channels", max_tokens, C);
#define RC(TT, V)                                                                                                              \
    PL_CUDA(launch_pdl(residual_conv_kernel<TT, V>, grid, block, 0, stream, (const TT*)h, C, cw, taps, state, state_stride, cu_q, \
                       slots, (TT*)out))
    if (dtype == PL_F32) {
        if (vec) RC(float, 4);
        else RC(float, 1);
    } else if (dtype == PL_BF16) {
        if (vec) RC(__nv_bfloat16, 4);
        else RC(__nv_bfloat16, 1);
    } else {
        return pl_fail("residual_conv: unknown dtype %d", dtype);
    }
#undef RC
    return 0;
}

// proj: [T, ld] in `dtype`, columns [r: C | k: C | v: C | g: C | removal: C | decay: rank] with C = H * d.  For few tokens per
// request; the norm of each head's output and the gate are part of it: out [T, C] in `dtype`.
PL_EXPORT int pl_general_delta_step(const void* proj, int dtype, int ld, const void* w_decay, int rank, const float* w0, const float* a_bias,
                                    int H, int d, float decay_scale, float unit_eps, const float* norm_w, float eps, float* state,
                                    long long state_stride, const int* cu_q, const int* slots, int num_seqs, void* out,
                                    cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    PL_REQUIRE(H > 0 && d > 0 && d <= 128 && rank > 0 && rank % 8 == 0 && rank <= GD_MAX_RANK && ld >= 5 * H * d + rank,
               "general_delta_step: bad sizes H=%d d=%d (at most 128) rank=%d ld=%d", H, d, rank, ld);
    PL_REQUIRE(((uintptr_t)w_decay & 15) == 0 && (long long)num_seqs * H < (1ll << 31), "general_delta_step: misaligned weights or too many blocks");
    const GdIn in = {proj, ld, w0, a_bias, H, d, decay_scale, unit_eps};
    const GdTail tail = {w_decay, rank, norm_w, eps};
    if (dtype == PL_F32) return launch_gd_step<float>(in, tail, state, state_stride, cu_q, slots, num_seqs, out, stream);
    if (dtype == PL_BF16) return launch_gd_step<__nv_bfloat16>(in, tail, state, state_stride, cu_q, slots, num_seqs, out, stream);
    return pl_fail("general_delta_step: unknown dtype %d", dtype);
}

// Scratch floats of pl_general_delta_chunks per (chunk, head); a step of T tokens and S requests takes T / pl_general_delta_chunk() + S
// chunks at most.
PL_EXPORT int pl_general_delta_chunk() { return GC; }
PL_EXPORT long long pl_general_delta_chunk_floats(int d) { return (long long)gc_floats(d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256); }

// Any number of tokens per request.  z: [T, C] float32, the decay's input in front of its bias; buf: scratch (16-byte aligned);
// out: [T, C] float32, the recurrence's output in front of the norm.
PL_EXPORT int pl_general_delta_chunks(const void* proj, int dtype, int ld, const float* z, const float* w0, const float* a_bias, int H, int d,
                                      float decay_scale, float unit_eps, float* buf, int max_chunks, float* state, long long state_stride,
                                      const int* cu_q, const int* slots, int num_seqs, float* out, cudaStream_t stream) {
    if (num_seqs == 0 || max_chunks == 0) return 0;
    PL_REQUIRE(H > 0 && d > 0 && d <= 256 && ld >= 5 * H * d, "general_delta_chunks: bad sizes H=%d d=%d ld=%d (key size at most 256)", H, d, ld);
    PL_REQUIRE(decay_scale <= 0.f && decay_scale >= -4.f, "general_delta_chunks: decay_scale=%g outside -4 .. 0 (1 / P would leave float32's range)",
               (double)decay_scale);
    PL_REQUIRE(((uintptr_t)buf & 15) == 0, "general_delta_chunks: misaligned scratch");
    const GdIn in = {proj, ld, w0, a_bias, H, d, decay_scale, unit_eps};
#define GDC(TT)                                                                                                                              \
    do {                                                                                                                                     \
        if (d <= 32) return launch_gd_chunks<TT, 32>(in, z, buf, max_chunks, state, state_stride, cu_q, slots, num_seqs, out, stream);       \
        if (d <= 64) return launch_gd_chunks<TT, 64>(in, z, buf, max_chunks, state, state_stride, cu_q, slots, num_seqs, out, stream);       \
        if (d <= 128) return launch_gd_chunks<TT, 128>(in, z, buf, max_chunks, state, state_stride, cu_q, slots, num_seqs, out, stream);     \
        return launch_gd_chunks<TT, 256>(in, z, buf, max_chunks, state, state_stride, cu_q, slots, num_seqs, out, stream);                   \
    } while (0)
    if (dtype == PL_F32) GDC(float);
    if (dtype == PL_BF16) GDC(__nv_bfloat16);
#undef GDC
    return pl_fail("general_delta_chunks: unknown dtype %d", dtype);
}
