// The generalized delta rule: a matrix state per head with a decay and a removal rate per key channel.
//
//     S <- diag(w) S - (a u) (u^T S) + k v^T,   o = S^T r          u = k / sqrt(sum k^2 + unit_eps), both terms from the old S
//     w = exp(decay_scale * sigmoid(z + w0)),   a = sigmoid(removal + removal bias)
//
// and the causal convolution per channel that is added to a mixer's input.  Everything is float32 whatever the
// activations' type is; the state of a request lives in a slot of [slots, state_stride] floats, a head's state column by
// column ([H][d][d], column j the d numbers S[:, j]).  The recurrence runs in the order of the tokens with a fixed order of
// sums, so what a position gets does not depend on how the prompt was cut or on the batch.
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

// ------------------------------------------------------------------ what does not depend on the state
// Per token and head, float32: vec[6][d] = [w | u | a u | k | r w | v] and scal[2] = [r . (a u) | r . k].  A warp computes
// one (token, head); `lane` takes channels lane, lane + 32, ...  proj row: [r: C | k: C | v: C | ... | removal: C at a_col].
struct GdIn {
    const void* proj;
    int ld, a_col;              // row stride, first column of the removal rates
    const float* z;             // [T, C]: the decay's input in front of its bias
    const float *w0, *a_bias;   // [C]
    int H, d;
    float decay_scale, unit_eps;
};

template <typename T>
__device__ __forceinline__ void gd_prepare(const GdIn& in, long long t, int h, int lane, float* w, float* u, float* au, float* k, float* rw,
                                           float* v, float* scal) {
    const int d = in.d, C = in.H * d, c0 = h * d;
    const T* row = (const T*)in.proj + (size_t)t * in.ld;
    float sq = 0.f;
    for (int i = lane; i < d; i += 32) {
        const float kv = to_float(row[C + c0 + i]);
        sq = fmaf(kv, kv, sq);
    }
    const float f = 1.0f / sqrtf(warp_sum(sq) + in.unit_eps);
    float rau = 0.f, rk = 0.f;
    for (int i = lane; i < d; i += 32) {
        const float rv = to_float(row[c0 + i]), kv = to_float(row[C + c0 + i]);
        const float a = sigmoid_f(to_float(row[in.a_col + c0 + i]) + __ldg(in.a_bias + c0 + i));
        const float wv = expf(in.decay_scale * sigmoid_f(in.z[(size_t)t * C + c0 + i] + __ldg(in.w0 + c0 + i)));
        const float uv = kv * f, auv = a * uv;
        w[i] = wv, u[i] = uv, au[i] = auv, k[i] = kv, rw[i] = rv * wv, v[i] = to_float(row[2 * C + c0 + i]);
        rau = fmaf(rv, auv, rau);
        rk = fmaf(rv, kv, rk);
    }
    rau = warp_sum(rau);
    rk = warp_sum(rk);
    if (lane == 0) scal[0] = rau, scal[1] = rk;
}

template <typename T>
__global__ void __launch_bounds__(256) gd_prepare_kernel(GdIn in, float* __restrict__ vec, float* __restrict__ scal, long long items) {
    const long long item = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (item >= items) return;
    const long long t = item / in.H;
    const int h = (int)(item - t * in.H), d = in.d;
    float* o = vec + (size_t)item * 6 * d;
    gd_prepare<T>(in, t, h, threadIdx.x & 31, o, o + d, o + 2 * d, o + 3 * d, o + 4 * d, o + 5 * d, scal + item * 2);
}

// ------------------------------------------------------------------ the recurrence
// grid: (requests, heads, blocks of COLS = 128 / LANES columns).  LANES lanes share a column of a head's state, lane l
// holding the key channels 4 l + 4 LANES m + (0..3), m < NPER / 4, in registers.  Per token, with the dots summed over the
// lanes by one butterfly:
//     c = u . S_j,  e = (r w) . S_j,  S_j <- w S_j - (a u) c + k v_j,  o_j = e - (r . a u) c + (r . k) v_j
// The vectors of TOK tokens at a time are staged in shared memory, the next ones by cp.async while these are worked on
// (PRE: they come prepared from global memory), or are formed right here (a step of few tokens per request).
constexpr int GD_THREADS = 128, GD_TOK = 8;

__device__ __forceinline__ void gd_cp4(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
                 "r"(ok ? 4 : 0));
}
__device__ __forceinline__ void gd_cp16(float* dst, const float* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src),
                 "r"(ok ? 16 : 0));
}

// Floats of one staging buffer: per token six rows of DP and two numbers.
__host__ __device__ constexpr int gd_stage_floats(int DP) { return GD_TOK * (6 * DP + 4); }

template <typename T, int NPER, int LANES, bool PRE>
__global__ void __launch_bounds__(GD_THREADS) gd_scan_kernel(GdIn in, const float* __restrict__ vec, const float* __restrict__ scal,
                                                             float* __restrict__ state, long long state_stride,
                                                             const int* __restrict__ cu_q, const int* __restrict__ slots,
                                                             float* __restrict__ out, int vec16) {
    constexpr int DP = NPER * LANES, COLS = GD_THREADS / LANES, STAGE = gd_stage_floats(DP), ROW = 6 * DP + 4;
    extern __shared__ __align__(16) float gd_smem[];
    const int s = blockIdx.x, h = blockIdx.y, d = in.d, H = in.H;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    if (slot < 0 || nq <= 0) return;
    const int tid = threadIdx.x, lane = tid % LANES, j = blockIdx.z * COLS + tid / LANES;
    const bool live = j < d;
    float* sp = state + (size_t)slot * state_stride + ((size_t)h * d + (live ? j : 0)) * d;
    float S[NPER];
#pragma unroll
    for (int r = 0; r < NPER; ++r) {
        const int ch = (r >> 2) * (4 * LANES) + lane * 4 + (r & 3);
        S[r] = live && ch < d ? sp[ch] : 0.f;
    }
    if (!PRE) {
        // the padding of the rows is zero for good
        for (int e = tid; e < STAGE; e += GD_THREADS) gd_smem[e] = 0.f;
        __syncthreads();
    }
    auto stage = [&](int t0, int buf) {
        float* base = gd_smem + buf * STAGE;
        const int nt = min(GD_TOK, nq - t0);
        if (!PRE) {
            for (int tt = tid >> 5; tt < nt; tt += GD_THREADS / 32) {
                float* o = base + tt * ROW;
                gd_prepare<T>(in, q0 + t0 + tt, h, tid & 31, o, o + DP, o + 2 * DP, o + 3 * DP, o + 4 * DP, o + 5 * DP, o + 6 * DP);
            }
            return;
        }
        const size_t first = ((size_t)(q0 + t0) * H + h), step = (size_t)H;
        if (vec16) {
            constexpr int CHUNKS = 6 * DP / 4;
            for (int e = tid; e < nt * CHUNKS; e += GD_THREADS) {
                const int tt = e / CHUNKS, q = e - tt * CHUNKS, which = q / (DP / 4), ch = (q - which * (DP / 4)) * 4;
                const bool ok = ch < d;
                gd_cp16(base + tt * ROW + which * DP + ch, vec + (first + tt * step) * 6 * d + (ok ? which * d + ch : 0), ok);
            }
        } else {
            for (int e = tid; e < nt * 6 * DP; e += GD_THREADS) {
                const int tt = e / (6 * DP), q = e - tt * (6 * DP), which = q / DP, ch = q - which * DP;
                const bool ok = ch < d;
                gd_cp4(base + tt * ROW + which * DP + ch, vec + (first + tt * step) * 6 * d + (ok ? which * d + ch : 0), ok);
            }
        }
        if (tid < nt * 2) gd_cp4(base + (tid >> 1) * ROW + 6 * DP + (tid & 1), scal + (first + (tid >> 1) * step) * 2 + (tid & 1), true);
    };
    stage(0, 0);
    if (PRE) asm volatile("cp.async.commit_group;\n" ::);
    int buf = 0;
    for (int t0 = 0; t0 < nq; t0 += GD_TOK) {
        const int nt = min(GD_TOK, nq - t0);
        if (PRE) {
            if (t0 + GD_TOK < nq) stage(t0 + GD_TOK, buf ^ 1);
            asm volatile("cp.async.commit_group;\n" ::);
            asm volatile("cp.async.wait_group 1;\n" ::);
        }
        __syncthreads();
        const float* base = gd_smem + buf * STAGE;
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float* row = base + tt * ROW;
            float c4[4] = {0.f, 0.f, 0.f, 0.f}, e4[4] = {0.f, 0.f, 0.f, 0.f};
            const float v = live ? row[5 * DP + j] : 0.f;
            const float rau = row[6 * DP], rk = row[6 * DP + 1];
#pragma unroll
            for (int m = 0; m < NPER / 4; ++m) {
                const float4 u4 = *reinterpret_cast<const float4*>(row + DP + m * (4 * LANES) + lane * 4);
                const float4 q4 = *reinterpret_cast<const float4*>(row + 4 * DP + m * (4 * LANES) + lane * 4);
                c4[0] = fmaf(S[4 * m], u4.x, c4[0]), c4[1] = fmaf(S[4 * m + 1], u4.y, c4[1]);
                c4[2] = fmaf(S[4 * m + 2], u4.z, c4[2]), c4[3] = fmaf(S[4 * m + 3], u4.w, c4[3]);
                e4[0] = fmaf(S[4 * m], q4.x, e4[0]), e4[1] = fmaf(S[4 * m + 1], q4.y, e4[1]);
                e4[2] = fmaf(S[4 * m + 2], q4.z, e4[2]), e4[3] = fmaf(S[4 * m + 3], q4.w, e4[3]);
            }
            float c = (c4[0] + c4[1]) + (c4[2] + c4[3]), e = (e4[0] + e4[1]) + (e4[2] + e4[3]);
            // One butterfly for both sums: after the first step the lower half of a column's lanes carries the partial
            // sums of c, the upper half those of e; c then goes to every lane from the column's first.
            const bool upper = lane >= LANES / 2;
            float x = upper ? e : c;
            x += __shfl_xor_sync(0xffffffffu, upper ? c : e, LANES / 2);
#pragma unroll
            for (int o = LANES / 4; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
            c = __shfl_sync(0xffffffffu, x, (tid & 31) & ~(LANES - 1));
#pragma unroll
            for (int m = 0; m < NPER / 4; ++m) {
                const float4 w4 = *reinterpret_cast<const float4*>(row + m * (4 * LANES) + lane * 4);
                const float4 a4 = *reinterpret_cast<const float4*>(row + 2 * DP + m * (4 * LANES) + lane * 4);
                const float4 k4 = *reinterpret_cast<const float4*>(row + 3 * DP + m * (4 * LANES) + lane * 4);
                S[4 * m] = fmaf(-a4.x, c, fmaf(w4.x, S[4 * m], k4.x * v));
                S[4 * m + 1] = fmaf(-a4.y, c, fmaf(w4.y, S[4 * m + 1], k4.y * v));
                S[4 * m + 2] = fmaf(-a4.z, c, fmaf(w4.z, S[4 * m + 2], k4.z * v));
                S[4 * m + 3] = fmaf(-a4.w, c, fmaf(w4.w, S[4 * m + 3], k4.w * v));
            }
            if (live && lane == LANES / 2) out[((size_t)(q0 + t0 + tt) * H + h) * d + j] = fmaf(rk, v, fmaf(-rau, c, x));
        }
        __syncthreads();                                            // the buffer is free again
        if (PRE) buf ^= 1;
        else if (t0 + GD_TOK < nq) stage(t0 + GD_TOK, 0);
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < NPER; ++r) {
            const int ch = (r >> 2) * (4 * LANES) + lane * 4 + (r & 3);
            if (ch < d) sp[ch] = S[r];
        }
    }
}

template <typename T, int NPER, bool PRE>
int launch_gd_scan(const GdIn& in, const float* vec, const float* scal, float* state, long long state_stride, const int* cu_q,
                   const int* slots, int num_seqs, float* out, cudaStream_t stream) {
    constexpr int LANES = 8, COLS = GD_THREADS / LANES;
    const dim3 grid(num_seqs, in.H, (in.d + COLS - 1) / COLS);
    PL_REQUIRE(grid.y <= 65535 && grid.z <= 65535, "general_delta: %d heads of %d", in.H, in.d);
    const size_t smem = (size_t)(PRE ? 2 : 1) * gd_stage_floats(NPER * LANES) * sizeof(float);
    auto kernel = gd_scan_kernel<T, NPER, LANES, PRE>;
    static bool opted = false;
    if (!opted && smem > 48 * 1024) {
        PL_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        opted = true;
    }
    kernel<<<grid, GD_THREADS, smem, stream>>>(in, vec, scal, state, state_stride, cu_q, slots, out,
                                               in.d % 4 == 0 && ((uintptr_t)vec & 15) == 0);
    PL_LAUNCHED("general_delta_scan");
    return 0;
}

template <typename T>
int general_delta(const GdIn& in, float* vec, float* scal, float* state, long long state_stride, const int* cu_q, const int* slots,
                  int num_seqs, long long tokens, float* out, cudaStream_t stream) {
    if (vec != nullptr) {
        const long long items = tokens * in.H, blocks = (items + 7) / 8;
        PL_REQUIRE(blocks < (1ll << 31), "general_delta: %lld tokens", tokens);
        gd_prepare_kernel<T><<<(unsigned)blocks, 256, 0, stream>>>(in, vec, scal, items);
        PL_LAUNCHED("general_delta_prepare");
    }
#define GD(N)                                                                                                                  \
    return vec != nullptr ? launch_gd_scan<T, N, true>(in, vec, scal, state, state_stride, cu_q, slots, num_seqs, out, stream) \
                          : launch_gd_scan<T, N, false>(in, vec, scal, state, state_stride, cu_q, slots, num_seqs, out, stream)
    if (in.d <= 32) GD(4);
    if (in.d <= 64) GD(8);
    if (in.d <= 128) GD(16);
    GD(32);
#undef GD
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

// proj: [T, ld] in `dtype`; z: [T, H*d] float32; out: [T, H*d] float32.  vec [T, H, 6, d] and scal [T, H, 2] float32: scratch for
// a kernel in front that forms what does not depend on the state, or null: the recurrence forms it itself (few tokens).
PL_EXPORT int pl_general_delta(const void* proj, int dtype, int ld, int a_col, const float* z, const float* w0, const float* a_bias,
                               int H, int d, float decay_scale, float unit_eps, float* vec, float* scal, float* state,
                               long long state_stride, const int* cu_q, const int* slots, int num_seqs, long long tokens, float* out,
                               cudaStream_t stream) {
    if (num_seqs == 0 || tokens == 0) return 0;
    PL_REQUIRE(H > 0 && d > 0 && d <= 256 && a_col >= 3 * H * d && a_col + H * d <= ld, "general_delta: bad sizes H=%d d=%d ld=%d (key size at most 256)",
               H, d, ld);
    PL_REQUIRE((vec == nullptr) == (scal == nullptr), "general_delta: half of the scratch is missing");
    const GdIn in = {proj, ld, a_col, z, w0, a_bias, H, d, decay_scale, unit_eps};
    if (dtype == PL_F32) return general_delta<float>(in, vec, scal, state, state_stride, cu_q, slots, num_seqs, tokens, out, stream);
    if (dtype == PL_BF16) return general_delta<__nv_bfloat16>(in, vec, scal, state, state_stride, cu_q, slots, num_seqs, tokens, out, stream);
    return pl_fail("general_delta: unknown dtype %d", dtype);
}
