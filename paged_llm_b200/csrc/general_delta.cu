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
constexpr int GD_MAX_RANK = 256, GS_THREADS = 256, GS_LANES = 8;

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

// Tokens of a request worked on at a time: a thread prepares one channel of one token.
__host__ __device__ constexpr int gs_tokens(int DP) { return GS_THREADS / DP; }
__host__ __device__ constexpr int gs_row(int DP) { return 6 * DP + 4; }
__host__ __device__ constexpr int gs_smem(int DP) {
    return (DP * DP + gs_tokens(DP) * (gs_row(DP) + DP + GD_MAX_RANK)) * (int)sizeof(float);
}

// The sum over a token's DP channels of two numbers per thread, in a fixed order, for all of the token's threads.
// red: [2][GS_THREADS / 32]; all threads of the block take part.
template <int DP>
__device__ __forceinline__ float2 gs_token_sum(float a, float b, float* red, int tid) {
    a = warp_sum(a), b = warp_sum(b);
    if (DP == 32) return make_float2(a, b);
    constexpr int W = DP / 32, NW = GS_THREADS / 32;
    if ((tid & 31) == 0) red[tid >> 5] = a, red[NW + (tid >> 5)] = b;
    __syncthreads();
    const int w0 = (tid >> 5) / W * W;
    float2 s = make_float2(red[w0], red[NW + w0]);
#pragma unroll
    for (int i = 1; i < W; ++i) s.x += red[w0 + i], s.y += red[NW + w0 + i];
    return s;
}

template <typename T, int NPER>
__global__ void __launch_bounds__(GS_THREADS, 3) gd_step_kernel(GdIn in, GdTail tail, float* __restrict__ state, long long state_stride,
                                                                const int* __restrict__ cu_q, const int* __restrict__ slots,
                                                                T* __restrict__ out, int vec) {
    constexpr int DP = NPER * GS_LANES, ROW = gs_row(DP), TOK = gs_tokens(DP), NW = GS_THREADS / 32;
    extern __shared__ __align__(16) float gs_raw[];
    float* Ss = gs_raw;                                 // [DP columns][DP]: the head's state
    float* rows = Ss + DP * DP;                         // [TOK][ROW]: w, u, a u, k, r w, v, r . (a u), r . k
    float* os = rows + TOK * ROW;                       // [TOK][DP]: the head's outputs
    float* th = os + TOK * DP;                          // [TOK][GD_MAX_RANK]
    __shared__ float red[3][2 * NW];
    pdl_launch_dependents();
    const int s = blockIdx.x / in.H, h = blockIdx.x - s * in.H, d = in.d, C = in.H * d, c0 = h * d;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    const int tid = threadIdx.x, lane = tid % GS_LANES, col = tid / GS_LANES, wlane = tid & 31;
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
    // this thread's channel of its token: what is weights
    const int tt = tid / DP, i = tid - tt * DP;
    const bool real = i < d;
    const float w0 = real ? __ldg(in.w0 + c0 + i) : 0.f, ab = real ? __ldg(in.a_bias + c0 + i) : 0.f, nw = real ? __ldg(tail.norm_w + c0 + i) : 0.f;
    const T* w2 = (const T*)tail.w_decay + (size_t)(c0 + (real ? i : 0)) * tail.rank;
    const T* proj = (const T*)in.proj;
    pdl_wait();
    for (int t0 = 0; t0 < nq; t0 += TOK) {
        const int nt = min(TOK, nq - t0);
        const bool last = t0 + TOK >= nq, live = real && tt < nt;
        const T* row_in = proj + (size_t)(q0 + t0 + (tt < nt ? tt : 0)) * in.ld + c0 + (real ? i : 0);
        const float r = live ? to_float(row_in[0]) : 0.f, k = live ? to_float(row_in[C]) : 0.f, v = live ? to_float(row_in[2 * C]) : 0.f;
        const float g = to_float(row_in[3 * C]), rem = to_float(row_in[4 * C]);
        for (int e = tid; e < nt * tail.rank; e += GS_THREADS) {
            const int t = e / tail.rank, q = e - t * tail.rank;
            // (rounded as the activations of a product are)
            th[t * GD_MAX_RANK + q] = to_float(from_float<T>(tanhf(to_float(proj[(size_t)(q0 + t0 + t) * in.ld + 5 * C + q]))));
        }
        const float unit = 1.0f / sqrtf(gs_token_sum<DP>(k * k, 0.f, red[0], tid).x + in.unit_eps);
        __syncthreads();
        float z = 0.f;
        if (live) {
#pragma unroll 4
            for (int q = 0; q < tail.rank; q += 8) {
                float w8[8];
                gs_load8(w2 + q, w8);
                const float4 a4 = *reinterpret_cast<const float4*>(th + tt * GD_MAX_RANK + q), b4 = *reinterpret_cast<const float4*>(th + tt * GD_MAX_RANK + q + 4);
                z = fmaf(a4.x, w8[0], z), z = fmaf(a4.y, w8[1], z), z = fmaf(a4.z, w8[2], z), z = fmaf(a4.w, w8[3], z);
                z = fmaf(b4.x, w8[4], z), z = fmaf(b4.y, w8[5], z), z = fmaf(b4.z, w8[6], z), z = fmaf(b4.w, w8[7], z);
            }
        }
        const float w = expf(in.decay_scale * sigmoid_f(z + w0)), u = k * unit, au = sigmoid_f(rem + ab) * u;
        float* row = rows + tt * ROW;                   // (channels that pad a row: everything but w is zero, and so is S)
        row[i] = w, row[DP + i] = u, row[2 * DP + i] = au, row[3 * DP + i] = k, row[4 * DP + i] = r * w, row[5 * DP + i] = v;
        const float2 dots = gs_token_sum<DP>(r * au, r * k, red[1], tid);
        if (i == 0) row[6 * DP] = dots.x, row[6 * DP + 1] = dots.y;
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();
#pragma unroll 2
        for (int j = col; j < DP; j += GS_THREADS / GS_LANES) {       // (uniform per warp: a multiple of its four columns)
            float S[NPER];
            const int jr = j < d ? j : 0;
#pragma unroll
            for (int m = 0; m < NPER / 4; ++m) {
                const float4 x = *reinterpret_cast<const float4*>(Ss + jr * DP + m * 32 + lane * 4);
                S[4 * m] = x.x, S[4 * m + 1] = x.y, S[4 * m + 2] = x.z, S[4 * m + 3] = x.w;
            }
            for (int t = 0; t < nt; ++t) {
                const float* ro = rows + t * ROW;
                const float rau = ro[6 * DP], rk = ro[6 * DP + 1], vj = ro[5 * DP + jr];
                float c4[4] = {0.f, 0.f, 0.f, 0.f}, e4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int m = 0; m < NPER / 4; ++m) {
                    const float4 u4 = *reinterpret_cast<const float4*>(ro + DP + m * 32 + lane * 4);
                    const float4 q4 = *reinterpret_cast<const float4*>(ro + 4 * DP + m * 32 + lane * 4);
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
                    const float4 w4 = *reinterpret_cast<const float4*>(ro + m * 32 + lane * 4);
                    const float4 a4 = *reinterpret_cast<const float4*>(ro + 2 * DP + m * 32 + lane * 4);
                    const float4 k4 = *reinterpret_cast<const float4*>(ro + 3 * DP + m * 32 + lane * 4);
                    S[4 * m] = fmaf(-a4.x, c, fmaf(w4.x, S[4 * m], k4.x * vj));
                    S[4 * m + 1] = fmaf(-a4.y, c, fmaf(w4.y, S[4 * m + 1], k4.y * vj));
                    S[4 * m + 2] = fmaf(-a4.z, c, fmaf(w4.z, S[4 * m + 2], k4.z * vj));
                    S[4 * m + 3] = fmaf(-a4.w, c, fmaf(w4.w, S[4 * m + 3], k4.w * vj));
                }
                if (lane == GS_LANES / 2) os[t * DP + j] = j < d ? fmaf(rk, vj, fmaf(-rau, c, x)) : 0.f;
            }
            if (j < d) {
#pragma unroll
                for (int m = 0; m < NPER / 4; ++m) {
                    const int ch = m * 32 + lane * 4;
                    const float4 x = make_float4(S[4 * m], S[4 * m + 1], S[4 * m + 2], S[4 * m + 3]);
                    if (!last) *reinterpret_cast<float4*>(Ss + j * DP + ch) = x;
                    else if (vec) {
                        if (ch < d) *reinterpret_cast<float4*>(sp + (size_t)j * d + ch) = x;
                    } else {
#pragma unroll
                        for (int q = 0; q < 4; ++q)
                            if (ch + q < d) sp[(size_t)j * d + ch + q] = S[4 * m + q];
                    }
                }
            }
        }
        __syncthreads();
        const float o = tt < nt ? os[tt * DP + i] : 0.f;
        const float f = 1.0f / sqrtf(gs_token_sum<DP>(o * o, 0.f, red[2], tid).x / (float)d + tail.eps);
        if (live) out[(size_t)(q0 + t0 + tt) * C + c0 + i] = from_float<T>(o * f * nw * sigmoid_f(g));
        if (!last) __syncthreads();
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

// A (chunk, head) in memory, in floats: the matrix above, row-major, a row GC_LD(DP) long (4 floats more than it needs, so that
// the second kernel's reads of eight rows meet no bank of shared memory twice); [2 GC][DP] what is added to the state per value
// and per c; [DP] P_end; the values, by blocks of 16 columns, [DP / 16][GC][16].
__host__ __device__ constexpr int gc_ld(int DP) { return DP + GC + 4; }
__host__ __device__ constexpr int gc_fixed(int DP) { return 2 * GC * gc_ld(DP) + 2 * GC * DP + DP; }
__host__ __device__ constexpr size_t gc_floats(int DP) { return (size_t)gc_fixed(DP) + GC * DP; }
__host__ __device__ constexpr int gc_prepare_smem(int DP) { return (4 * GC * (DP + 4) + 4 * GC * GC + GC) * (int)sizeof(float); }

template <typename T, int DP>
__global__ void __launch_bounds__(GC_THREADS, DP <= 128 ? 4 : 1) gd_chunk_prepare_kernel(GdIn in, const float* __restrict__ z, const int* __restrict__ cu_q,
                                                                      const int* __restrict__ slots, int num_seqs, float* __restrict__ buf) {
    constexpr int LD = DP + 4;                          // rows 4 floats longer: 16-byte reads of eight rows meet no bank twice
    constexpr int PARTS = GC_THREADS / DP, TP = GC / PARTS;          // threads per channel, tokens of each
    extern __shared__ __align__(16) float gc_smem[];
    float *xs = gc_smem, *bs = xs + GC * LD, *ks = bs + GC * LD, *ys = ks + GC * LD;      // first w, a, k, r; then x, b, k~, y
    float* gram = ys + GC * LD;                         // [x . k~ | x . b | y . k~ | y . b][s][t]: a column of each in a row
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
    float* M = buf + ((size_t)chunk * in.H + h) * gc_floats(DP);
    float* W = M + 2 * GC * gc_ld(DP);
    float* Pend = W + 2 * GC * DP;
    float* V = Pend + DP;
    // a thread per channel and PARTS apart in the tokens, all loads of a token independent of each other
    {
        const int i = tid % DP;
        const bool real = i < d;
        const float w0 = real ? __ldg(in.w0 + c0 + i) : 0.f, ab = real ? __ldg(in.a_bias + c0 + i) : 0.f;
#pragma unroll 4
        for (int t = tid / DP; t < GC; t += PARTS) {
            float w = 1.f, a = 0.f, k = 0.f, r = 0.f, v = 0.f;
            if (t < nt && real) {
                const T* row = row0 + (size_t)t * in.ld + i;
                r = to_float(row[0]), k = to_float(row[C]), v = to_float(row[2 * C]);
                w = expf(in.decay_scale * sigmoid_f(z0[(size_t)t * C + i] + w0));
                a = sigmoid_f(to_float(row[4 * C]) + ab);
            }
            xs[t * LD + i] = w, bs[t * LD + i] = a, ks[t * LD + i] = k, ys[t * LD + i] = r;
            V[(i >> 4) * (GC * 16) + t * 16 + (i & 15)] = v;
        }
    }
    __syncthreads();
#pragma unroll
    for (int t = warp; t < GC; t += GC_THREADS / 32) {
        float sq = 0.f;
#pragma unroll
        for (int i = lane; i < DP; i += 32) sq = fmaf(ks[t * LD + i], ks[t * LD + i], sq);
        sq = warp_sum(sq);
        if (lane == 0) unit[t] = 1.0f / sqrtf(sq + in.unit_eps);
    }
    float P = 1.f, total = 1.f, ws[TP];
    const int ci = tid % DP, ct0 = tid / DP * TP;
#pragma unroll
    for (int t = 0; t < GC; ++t) {
        const float w = xs[t * LD + ci];
        if (t == ct0) P = total;
        total *= w;
    }
#pragma unroll
    for (int t = 0; t < TP; ++t) ws[t] = xs[(ct0 + t) * LD + ci];
    __syncthreads();                                    // (`unit`, and every w is read)
    if (ct0 == 0) Pend[ci] = total;
#pragma unroll
    for (int q = 0; q < TP; ++q) {
        const int t = ct0 + q;
        const float k = ks[t * LD + ci], u = k * unit[t], au = bs[t * LD + ci] * u;
        xs[t * LD + ci] = P * u;
        P *= ws[q];
        const float inv = 1.0f / P, kk = k * inv, b = au * inv;
        bs[t * LD + ci] = b;
        ks[t * LD + ci] = kk;
        ys[t * LD + ci] *= P;
        W[t * DP + ci] = kk * total;
        W[(GC + t) * DP + ci] = -b * total;
    }
    __syncthreads();
    {
        // a thread per pair (t, s): four dots
        const int q = tid / GC, t = tid - q * GC;
        float xk = 0.f, xb = 0.f, yk = 0.f, yb = 0.f;
#pragma unroll 4
        for (int i = 0; i < DP; i += 4) {
            const float4 x = *reinterpret_cast<const float4*>(xs + t * LD + i), y = *reinterpret_cast<const float4*>(ys + t * LD + i);
            const float4 k = *reinterpret_cast<const float4*>(ks + q * LD + i), b = *reinterpret_cast<const float4*>(bs + q * LD + i);
            xk = fmaf(x.x, k.x, fmaf(x.y, k.y, fmaf(x.z, k.z, fmaf(x.w, k.w, xk))));
            xb = fmaf(x.x, b.x, fmaf(x.y, b.y, fmaf(x.z, b.z, fmaf(x.w, b.w, xb))));
            yk = fmaf(y.x, k.x, fmaf(y.y, k.y, fmaf(y.z, k.z, fmaf(y.w, k.w, yk))));
            yb = fmaf(y.x, b.x, fmaf(y.y, b.y, fmaf(y.z, b.z, fmaf(y.w, b.w, yb))));
        }
        gram[q * GC + t] = q < t ? xk : 0.f;
        gram[GC * GC + q * GC + t] = q < t ? xb : 0.f;
        gram[2 * GC * GC + q * GC + t] = q <= t ? yk : 0.f;
        gram[3 * GC * GC + q * GC + t] = q <= t ? yb : 0.f;
    }
    __syncthreads();
    // forward substitution, a thread per column of [X | G] and the same column of [Y | H]: row by row, each solved entry is
    // taken out of all entries behind it
    for (int c = tid; c < DP + GC; c += GC_THREADS) {
        float x[GC], y[GC];
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            x[t] = c < DP ? xs[t * LD + c] : gram[(c - DP) * GC + t];
            y[t] = c < DP ? ys[t * LD + c] : gram[2 * GC * GC + (c - DP) * GC + t];
        }
#pragma unroll
        for (int q = 0; q < GC; ++q) {
            const float* xb = gram + GC * GC + q * GC;
            const float* yb = gram + 3 * GC * GC + q * GC;
#pragma unroll
            for (int t4 = q / 4 * 4; t4 < GC; t4 += 4) {
                const float4 a = *reinterpret_cast<const float4*>(xb + t4), b = *reinterpret_cast<const float4*>(yb + t4);
                if (t4 + 0 > q) x[t4 + 0] = fmaf(-a.x, x[q], x[t4 + 0]);
                if (t4 + 1 > q) x[t4 + 1] = fmaf(-a.y, x[q], x[t4 + 1]);
                if (t4 + 2 > q) x[t4 + 2] = fmaf(-a.z, x[q], x[t4 + 2]);
                if (t4 + 3 > q) x[t4 + 3] = fmaf(-a.w, x[q], x[t4 + 3]);
                if (t4 + 0 >= q) y[t4 + 0] = fmaf(-b.x, x[q], y[t4 + 0]);
                if (t4 + 1 >= q) y[t4 + 1] = fmaf(-b.y, x[q], y[t4 + 1]);
                if (t4 + 2 >= q) y[t4 + 2] = fmaf(-b.z, x[q], y[t4 + 2]);
                if (t4 + 3 >= q) y[t4 + 3] = fmaf(-b.w, x[q], y[t4 + 3]);
            }
        }
#pragma unroll
        for (int t = 0; t < GC; ++t) {
            M[(size_t)t * gc_ld(DP) + c] = x[t];
            M[(size_t)(GC + t) * gc_ld(DP) + c] = y[t];
        }
    }
}

// The second kernel's tiles: a thread owns GC_R rows x 4 columns of the state's block; the block's rows are so far apart that
// the reads of a warp's tiles meet no bank twice.
__host__ __device__ constexpr int gc_r(int DP) { return DP >= 64 ? DP / 64 : 1; }
__host__ __device__ constexpr int gc_sld(int DP) { return gc_r(DP) == 1 ? 16 : gc_r(DP) == 2 ? 24 : 20; }
// Its shared floats: two stages of [matrix | additions | P_end | a block of the values], the state's block of columns, c, and
// the partial sums of eight warps.
__host__ __device__ constexpr int gc_stage_floats(int DP) { return gc_fixed(DP) + GC * GC_COLS; }
__host__ __device__ constexpr int gc_scan_smem(int DP) {
    return (2 * gc_stage_floats(DP) + DP * gc_sld(DP) + GC * GC_COLS + 8 * 2 * GC * GC_COLS) * (int)sizeof(float);
}

template <int R>
__device__ __forceinline__ void gc_rows(const float* p, float (&w)[R]) {
    if (R == 2) {
        const float2 v = *reinterpret_cast<const float2*>(p);
        w[0] = v.x, w[R > 1 ? 1 : 0] = v.y;
    } else if (R == 4) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        w[0] = v.x, w[R > 1 ? 1 : 0] = v.y, w[R > 2 ? 2 : 0] = v.z, w[R > 3 ? 3 : 0] = v.w;
    } else {
        w[0] = p[0];
    }
}

// grid: (requests, heads, blocks of 16 columns); 256 threads.  Per chunk: the 2 GC x 16 product over the DP + GC rows of state
// and values, cut between the eight warps (tiles of 4 x 4 per thread) and summed in a fixed order; then the state's update,
// whose part that does not wait for the sums runs in front of them.
template <int DP>
__global__ void __launch_bounds__(GC_THREADS) gd_chunk_scan_kernel(int H, int d, const float* __restrict__ buf, float* __restrict__ state,
                                                                   long long state_stride, const int* __restrict__ cu_q,
                                                                   const int* __restrict__ slots, float* __restrict__ out) {
    constexpr int STAGE = gc_stage_floats(DP), FIXED = gc_fixed(DP), LDM = gc_ld(DP), SLD = gc_sld(DP), R = gc_r(DP);
    constexpr int QUADS = (DP + GC) / 4, BASE = QUADS / 8;           // quads of k: the first four warps take one more
    static_assert(QUADS == 8 * BASE + 4 && FIXED % 4 == 0, "");
    extern __shared__ __align__(16) float gc_smem_raw[];
    float* Ss = gc_smem_raw + 2 * STAGE;                // [DP][SLD]
    float* Cs = Ss + DP * SLD;                          // [GC][16]
    float* part = Cs + GC * GC_COLS;                    // [8 warps][4][32 lanes][4]
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
        for (int e = tid; e < FIXED / 4; e += GC_THREADS) gd_cp16(dst + e * 4, src + e * 4);
        if (tid < GC * GC_COLS / 4) gd_cp16(dst + FIXED + tid * 4, src + FIXED + (size_t)blockIdx.z * GC * GC_COLS + tid * 4);
        asm volatile("cp.async.commit_group;\n" ::);
    };
    stage(0, 0);
    for (int e = tid; e < GC_COLS * DP; e += GC_THREADS) {
        const int j = e / DP, k = e - j * DP;
        Ss[k * SLD + j] = j0 + j < d && k < d ? sp[(size_t)(j0 + j) * d + k] : 0.f;
    }
    const int rg = lane >> 2, ct = (lane & 3) * 4;                   // rows rg, rg + 8, .. of the product, columns ct .. ct + 3
    const int g_lo = warp * BASE + min(warp, 4), g_hi = g_lo + BASE + (warp < 4 ? 1 : 0);
    const int sr = (tid >> 2) * R, sc = ct;
    const bool owns = sr < DP;
    for (int c = 0; c < chunks; ++c) {
        const int b = c & 1, nt = min(GC, nq - c * GC);
        asm volatile("cp.async.wait_group 0;\n" ::);
        __syncthreads();
        if (c + 1 < chunks) stage(c + 1, b ^ 1);
        const float* M = gc_smem_raw + b * STAGE;
        const float* W = M + 2 * GC * LDM;
        const float* Pend = W + 2 * GC * DP;
        const float* V = Pend + DP;
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll
        for (int gi = 0; gi < BASE + 1; ++gi) {
            const int k4 = (g_lo + gi) * 4;
            if (gi == BASE && g_lo + gi >= g_hi) break;              // uniform per warp
            const float* xp = k4 < DP ? Ss + k4 * SLD + ct : V + (k4 - DP) * GC_COLS + ct;
            const int xs = k4 < DP ? SLD : GC_COLS;
            float4 m[4], x[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                m[i] = *reinterpret_cast<const float4*>(M + (rg + 8 * i) * LDM + k4);
                x[i] = *reinterpret_cast<const float4*>(xp + i * xs);
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float mm[4] = {m[i].x, m[i].y, m[i].z, m[i].w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    acc[i][0] = fmaf(mm[k], x[k].x, acc[i][0]), acc[i][1] = fmaf(mm[k], x[k].y, acc[i][1]);
                    acc[i][2] = fmaf(mm[k], x[k].z, acc[i][2]), acc[i][3] = fmaf(mm[k], x[k].w, acc[i][3]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
            *reinterpret_cast<float4*>(part + ((warp * 4 + i) * 32 + lane) * 4) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        // what does not wait for c: the decayed state and the values' part
        float st[R][4];
        if (owns) {
            float p[R];
            gc_rows<R>(Pend + sr, p);
#pragma unroll
            for (int r = 0; r < R; ++r) {
                const float4 x = *reinterpret_cast<const float4*>(Ss + (sr + r) * SLD + sc);
                st[r][0] = p[r] * x.x, st[r][1] = p[r] * x.y, st[r][2] = p[r] * x.z, st[r][3] = p[r] * x.w;
            }
#pragma unroll 8
            for (int q = 0; q < GC; ++q) {
                const float4 x = *reinterpret_cast<const float4*>(V + q * GC_COLS + sc);
                float w[R];
                gc_rows<R>(W + q * DP + sr, w);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    st[r][0] = fmaf(w[r], x.x, st[r][0]), st[r][1] = fmaf(w[r], x.y, st[r][1]);
                    st[r][2] = fmaf(w[r], x.z, st[r][2]), st[r][3] = fmaf(w[r], x.w, st[r][3]);
                }
            }
        }
        __syncthreads();
        {
            const int i = tid >> 6, l = (tid >> 1) & 31, half = (tid & 1) * 2;
            const int row = (l >> 2) + 8 * i, col = (l & 3) * 4 + half;
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int w = 0; w < 8; ++w) {
                const float2 x = *reinterpret_cast<const float2*>(part + ((w * 4 + i) * 32 + l) * 4 + half);
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
#pragma unroll 8
            for (int q = 0; q < GC; ++q) {
                const float4 x = *reinterpret_cast<const float4*>(Cs + q * GC_COLS + sc);
                float w[R];
                gc_rows<R>(W + (GC + q) * DP + sr, w);
#pragma unroll
                for (int r = 0; r < R; ++r) {
                    st[r][0] = fmaf(w[r], x.x, st[r][0]), st[r][1] = fmaf(w[r], x.y, st[r][1]);
                    st[r][2] = fmaf(w[r], x.z, st[r][2]), st[r][3] = fmaf(w[r], x.w, st[r][3]);
                }
            }
#pragma unroll
            for (int r = 0; r < R; ++r)
                *reinterpret_cast<float4*>(Ss + (sr + r) * SLD + sc) = make_float4(st[r][0], st[r][1], st[r][2], st[r][3]);
        }
    }
    __syncthreads();
    for (int e = tid; e < GC_COLS * DP; e += GC_THREADS) {
        const int j = e / DP, k = e - j * DP;
        if (j0 + j < d && k < d) sp[(size_t)(j0 + j) * d + k] = Ss[k * SLD + j];
    }
}

template <typename T, int DP>
int launch_gd_chunks(const GdIn& in, const float* z, float* buf, int slots_of_chunks, float* state, long long state_stride, const int* cu_q,
                     const int* slots, int num_seqs, float* out, cudaStream_t stream) {
    static bool opted = false;
    if (!opted) {
        PL_CUDA(cudaFuncSetAttribute(gd_chunk_prepare_kernel<T, DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, gc_prepare_smem(DP)));
        PL_CUDA(cudaFuncSetAttribute(gd_chunk_prepare_kernel<T, DP>, cudaFuncAttributePreferredSharedMemoryCarveout, (int)cudaSharedmemCarveoutMaxShared));
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
