// Linear attention with a fixed decay per head ("Lightning Attention-2", Qin et al.), in float32 state:
//
//     q = silu(.), k = silu(.), v = silu(.)            (the projection's columns, rounded to the compute type)
//     S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
//
// and the norm over a row of all heads together, times the sigmoid of a gate.
//
// proj: rows [q: H*d | k: H*d | v: H*dv | ...] with row stride ld in the compute type; state: [H][dv][d] floats per slot (a
// head's columns one after the other); o: [T, H*dv] float32.  Two forms:
//
//  * token by token (decoding, short portions, float32): every lane keeps its part of a few columns in registers and the
//    sums are float32 multiply-adds in a fixed order;
//  * in chunks of LC tokens (bfloat16 prompt portions): what a chunk adds to the state is one product per chunk, the states
//    at the chunks' starts follow from those by a scan over chunks, and the outputs of a chunk are
//        o_i = decay^(i+1) S_start^T q_i + sum_{j <= i} decay^(i-j) (q_i . k_j) v_j.
//    The products run on the tensor cores (mma.sync).  q, k and v are bfloat16 already (silu is applied in place by a kernel
//    in front); every operand that is not (the state, the decayed values, the decayed scores) is split into two bfloat16
//    parts, x = hi + lo, whose products are both added in float32.
#include "common.cuh"

namespace {

constexpr int LC = 128;         // tokens of a chunk
constexpr int LH = 64;          // tokens worked on at once

// silu as the compute type holds it.  Before the rounding to bfloat16 the quick exponential and division are exact enough.
template <typename T> __device__ __forceinline__ float rounded_silu(float x);
template <> __device__ __forceinline__ float rounded_silu<float>(float x) { return silu_f(x); }
template <> __device__ __forceinline__ float rounded_silu<__nv_bfloat16>(float x) {
    return __bfloat162float(__float2bfloat16_rn(__fdividef(x, 1.0f + __expf(fminf(-x, 80.f)))));
}

// ------------------------------------------------------------------ token by token
// grid: (requests, heads, blocks of columns).  LPC lanes share a column, each holding NV float4 of its key channels (lane l:
// channels 4 l + 4 LPC i ..+3); a warp has 32 / LPC columns side by side and R of those rows.
template <typename T, int LPC, int NV, int R>
__global__ void __launch_bounds__(256) lightning_step_kernel(const T* __restrict__ proj, int ld, int H, int d, int dv,
                                                             const float* __restrict__ decay, float* __restrict__ state,
                                                             long long state_stride, const int* __restrict__ cu_q,
                                                             const int* __restrict__ slots, float* __restrict__ o, int vec) {
    constexpr int CPW = 32 / LPC;
    pdl_launch_dependents();
    const int s = blockIdx.x, h = blockIdx.y;
    const int slot = slots[s];
    const int q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, sub = lane / LPC, l = lane % LPC;
    const int v0 = (blockIdx.z * 8 + warp) * (R * CPW) + sub;           // column of row r: v0 + r * CPW
    if (slot < 0 || nq <= 0) {
        pdl_wait();
        return;
    }
    const float dec = __ldg(decay + h);
    float* st = state + (size_t)slot * state_stride + (size_t)h * dv * d;
    float S[R][NV * 4];
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int v = v0 + r * CPW, n = 4 * l + 4 * LPC * i;
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (v < dv && n < d) {
                const float* p = st + (size_t)v * d + n;
                if (vec) {
                    x = *reinterpret_cast<const float4*>(p);
                } else {
                    x.x = p[0];
                    if (n + 1 < d) x.y = p[1];
                    if (n + 2 < d) x.z = p[2];
                    if (n + 3 < d) x.w = p[3];
                }
            }
            S[r][4 * i] = x.x, S[r][4 * i + 1] = x.y, S[r][4 * i + 2] = x.z, S[r][4 * i + 3] = x.w;
        }
    pdl_wait();
    const int kcol = H * d + h * d, vcol = 2 * H * d + h * dv;
    for (int t = 0; t < nq; ++t) {
        const T* row = proj + (size_t)(q0 + t) * ld;
        float q[NV * 4], k[NV * 4], acc[R];
#pragma unroll
        for (int i = 0; i < NV * 4; ++i) {
            const int n = 4 * l + 4 * LPC * (i >> 2) + (i & 3);
            q[i] = n < d ? rounded_silu<T>(to_float(row[h * d + n])) : 0.f;
            k[i] = n < d ? rounded_silu<T>(to_float(row[kcol + n])) : 0.f;
        }
#pragma unroll
        for (int r = 0; r < R; ++r) {
            const int v = v0 + r * CPW;
            const float x = v < dv ? rounded_silu<T>(to_float(row[vcol + v])) : 0.f;
            float a = 0.f;
#pragma unroll
            for (int i = 0; i < NV * 4; ++i) {
                S[r][i] = fmaf(dec, S[r][i], k[i] * x);
                a = fmaf(S[r][i], q[i], a);
            }
            acc[r] = a;
        }
        // The lanes' parts are summed by a butterfly that halves the rows a lane carries while there is more than one.
        int row_of = 0, n = R;
#pragma unroll
        for (int m = LPC / 2; m >= 1; m >>= 1) {
            if (n > 1) {
                n >>= 1;
                const bool upper = lane & m;
                row_of += upper ? n : 0;
#pragma unroll
                for (int i = 0; i < R / 2; ++i)
                    if (i < n) {
                        const float send = upper ? acc[i] : acc[i + n], keep = upper ? acc[i + n] : acc[i];
                        acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                    }
            } else {
                acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], m);
            }
        }
        // (n rows are left in a lane: one, or several where a column has fewer lanes than rows)
        constexpr int LEFT = R > LPC ? R / LPC : 1, SAME = LPC > R ? LPC / R : 1;
        if (l % SAME == 0) {
#pragma unroll
            for (int i = 0; i < LEFT; ++i) {
                const int v = v0 + (row_of + i) * CPW;
                if (v < dv) o[(size_t)(q0 + t) * H * dv + (size_t)h * dv + v] = acc[i];
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int v = v0 + r * CPW, n = 4 * l + 4 * LPC * i;
            if (v < dv && n < d) {
                float* p = st + (size_t)v * d + n;
                if (vec) {
                    *reinterpret_cast<float4*>(p) = make_float4(S[r][4 * i], S[r][4 * i + 1], S[r][4 * i + 2], S[r][4 * i + 3]);
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (n + e < d) p[e] = S[r][4 * i + e];
                }
            }
        }
}

// ------------------------------------------------------------------ in chunks
// Chunks are numbered so that a request's chunks follow each other and every request has room: chunk c of request s is
// cu_q[s] / LC + s + c.  The block of a number finds its request by bisection.
struct ChunkAt {
    int s, c, q0, nq;           // request, its chunk, its first row, its tokens; s < 0: nobody's number
};

__device__ __forceinline__ ChunkAt find_chunk(const int* cu_q, int num_seqs, int number) {
    int lo = 0, hi = num_seqs;                                          // the last s with cu_q[s] / LC + s <= number
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (cu_q[mid] / LC + mid <= number) lo = mid; else hi = mid;
    }
    ChunkAt a;
    a.q0 = cu_q[lo], a.nq = cu_q[lo + 1] - a.q0;
    a.c = number - (a.q0 / LC + lo);
    a.s = a.c * LC < a.nq ? lo : -1;
    return a;
}

__device__ __forceinline__ void ldm4(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], const __nv_bfloat16* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
                 : "r"((uint32_t)__cvta_generic_to_shared(p)));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// x, y as packed bfloat16 (x in the lower half) and what the rounding left over.
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 r = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&r);
}

// silu of the first n columns of every row, in place.
__global__ void __launch_bounds__(256) lightning_silu_kernel(__nv_bfloat16* __restrict__ proj, int ld, int n, int rows, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    if (vec) {
        const int c = (blockIdx.x * 256 + threadIdx.x) * 8;
        if (c >= n) return;
        for (int r = blockIdx.y; r < rows; r += gridDim.y) {
            uint4* p = reinterpret_cast<uint4*>(proj + (size_t)r * ld + c);
            uint4 raw = *p;
            __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int i = 0; i < 4; ++i)
                h[i] = __floats2bfloat162_rn(rounded_silu<__nv_bfloat16>(__low2float(h[i])), rounded_silu<__nv_bfloat16>(__high2float(h[i])));
            *p = raw;
        }
        return;
    }
    for (int r = blockIdx.y; r < rows; r += gridDim.y)
        for (int c = blockIdx.x * 256 + threadIdx.x; c < n; c += gridDim.x * 256) {
            __nv_bfloat16* p = proj + (size_t)r * ld + c;
            *p = __float2bfloat16_rn(rounded_silu<__nv_bfloat16>(__bfloat162float(*p)));
        }
}

__device__ __forceinline__ void cp16(__nv_bfloat16* dst, const __nv_bfloat16* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0));
}
__device__ __forceinline__ void cp_done() {
    asm volatile("cp.async.commit_group;\n" ::);
    asm volatile("cp.async.wait_group 0;\n" ::);
}

// A tile of `rows` rows and `cols` columns (a multiple of 8) into shared memory with row stride `ds`, zeros behind the first
// `have_rows` rows and `have_cols` columns.  With `vec` by asynchronous copies of 16 bytes (cp_done), else element by element.
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, int ds, const __nv_bfloat16* src, size_t ld, int rows, int cols, int have_rows,
                                          int have_cols, int vec) {
    const int units = cols / 8;
    for (int e = threadIdx.x; e < rows * units; e += 128) {
        const int r = e / units, c = (e - r * units) * 8;
        if (vec) {
            const bool in = r < have_rows && c < have_cols;
            cp16(dst + r * ds + c, src + (in ? (size_t)r * ld + c : 0), in);
        } else {
#pragma unroll
            for (int i = 0; i < 8; ++i)
                dst[r * ds + c + i] = r < have_rows && c + i < have_cols ? src[(size_t)r * ld + c + i] : __float2bfloat16_rn(0.f);
        }
    }
}

// What chunk c adds to the state by its end: add[number][h][v][n] = sum_j decay^(len-1-j) v_j[v] k_j[n].  grid: (numbers,
// heads, tiles of AV values x AK key channels); four warps of 16 values each.
constexpr int AV = 64, AK = 128;

__global__ void __launch_bounds__(128) lightning_add_kernel(const __nv_bfloat16* __restrict__ proj, int ld, int H, int d, int dv, int dp,
                                                            const float* __restrict__ decay, const int* __restrict__ cu_q,
                                                            const int* __restrict__ slots, int num_seqs, float* __restrict__ add,
                                                            int vec) {
    __shared__ __align__(16) __nv_bfloat16 vh[LH][AV + 8], vl[LH][AV + 8], ks[LH][AK + 8];
    __shared__ float pw[LC];
    const ChunkAt at = find_chunk(cu_q, num_seqs, blockIdx.x);
    if (at.s < 0 || slots[at.s] < 0) return;
    const int h = blockIdx.y, ktiles = (dp + AK - 1) / AK;
    const int v0 = (blockIdx.z / ktiles) * AV, n0 = (blockIdx.z % ktiles) * AK;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int len = min(LC, at.nq - at.c * LC);
    const __nv_bfloat16* kb = proj + (size_t)(at.q0 + at.c * LC) * ld + H * d + h * d + n0;
    const __nv_bfloat16* vb = proj + (size_t)(at.q0 + at.c * LC) * ld + 2 * H * d + h * dv + v0;
    pw[tid] = powf(__ldg(decay + h), (float)tid);
    float acc[AK / 8][4];
#pragma unroll
    for (int i = 0; i < AK / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int t0 = 0; t0 < len; t0 += LH) {
        if (t0 > 0) __syncthreads();
        load_tile(&vh[0][0], AV + 8, vb + (size_t)t0 * ld, ld, LH, AV, len - t0, dv - v0, vec);
        load_tile(&ks[0][0], AK + 8, kb + (size_t)t0 * ld, ld, LH, AK, len - t0, d - n0, vec);
        cp_done();
        __syncthreads();
        for (int e = tid; e < LH * (AV / 8); e += 128) {                // the values times their decays, in two parts
            const int t = e / (AV / 8), c = (e % (AV / 8)) * 8;
            const float f = t0 + t < len ? pw[len - 1 - t0 - t] : 0.f;
            uint4 hi = *reinterpret_cast<const uint4*>(&vh[t][c]), lo;
            uint32_t* hw = reinterpret_cast<uint32_t*>(&hi);
            uint32_t* lw = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(hw + i);
                split_pair(__low2float(x) * f, __high2float(x) * f, hw[i], lw[i]);
            }
            *reinterpret_cast<uint4*>(&vh[t][c]) = hi;
            *reinterpret_cast<uint4*>(&vl[t][c]) = lo;
        }
        __syncthreads();
#pragma unroll
        for (int k0 = 0; k0 < LH; k0 += 16) {
            uint32_t a[4], a2[4];
            const int ar = k0 + (lane & 7) + (lane >= 16 ? 8 : 0), ac = warp * 16 + ((lane >> 3) & 1) * 8;
            ldm4t(a, &vh[ar][ac]);
            ldm4t(a2, &vl[ar][ac]);
#pragma unroll
            for (int n = 0; n < AK; n += 16) {
                uint32_t b[4];
                ldm4t(b, &ks[k0 + (lane & 7) + ((lane >> 3) & 1) * 8][n + (lane >= 16 ? 8 : 0)]);
                mma16816(acc[n / 8], a, b[0], b[1]);
                mma16816(acc[n / 8 + 1], a, b[2], b[3]);
                mma16816(acc[n / 8], a2, b[0], b[1]);
                mma16816(acc[n / 8 + 1], a2, b[2], b[3]);
            }
        }
    }
    float* out = add + ((size_t)blockIdx.x * H + h) * dv * dp;
#pragma unroll
    for (int i = 0; i < AK / 8; ++i) {
        const int n = n0 + i * 8 + (lane & 3) * 2, v = v0 + warp * 16 + (lane >> 2);
        if (n >= dp) continue;
        if (v < dv) *reinterpret_cast<float2*>(out + (size_t)v * dp + n) = make_float2(acc[i][0], acc[i][1]);
        if (v + 8 < dv) *reinterpret_cast<float2*>(out + (size_t)(v + 8) * dp + n) = make_float2(acc[i][2], acc[i][3]);
    }
}

// The states at the chunks' starts, as two parts of bfloat16: starts[number][h][hi, lo][v][n].  The state behind the last chunk
// goes to the request's slot.  A thread per four values.
__global__ void __launch_bounds__(256) lightning_scan_kernel(const float* __restrict__ add, __nv_bfloat16* __restrict__ starts, int H, int d,
                                                             int dv, int dp, const float* __restrict__ decay, const int* __restrict__ cu_q,
                                                             const int* __restrict__ slots, float* __restrict__ state,
                                                             long long state_stride, int vec) {
    const int s = blockIdx.x, h = blockIdx.y;
    const int slot = slots[s], q0 = cu_q[s], nq = cu_q[s + 1] - q0;
    const int e = (blockIdx.z * 256 + threadIdx.x) * 4;
    if (slot < 0 || nq <= 0 || e >= dv * dp) return;
    const int v = e / dp, n = e - v * dp;
    float* st = state + (size_t)slot * state_stride + ((size_t)h * dv + v) * d + n;
    float S[4] = {0.f, 0.f, 0.f, 0.f};
    if (vec && n < d) {
        const float4 x = *reinterpret_cast<const float4*>(st);
        S[0] = x.x, S[1] = x.y, S[2] = x.z, S[3] = x.w;
    } else {
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (n + i < d) S[i] = st[i];
    }
    const float dec = __ldg(decay + h), whole = powf(dec, (float)LC);
    const int chunks = (nq + LC - 1) / LC;
    const size_t step = (size_t)H * dv * dp, first = ((size_t)(q0 / LC + s) * H + h) * dv * dp;
    const float* p = add + first + e;
    __nv_bfloat16* w = starts + 2 * first + e;
    constexpr int AHEAD = 4;
    for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
        float4 more[AHEAD];
#pragma unroll
        for (int i = 0; i < AHEAD; ++i)
            if (c0 + i < chunks) more[i] = *reinterpret_cast<const float4*>(p + (size_t)(c0 + i) * step);
#pragma unroll
        for (int i = 0; i < AHEAD; ++i) {
            const int c = c0 + i;
            if (c >= chunks) break;
            uint2 hi, lo;
            split_pair(S[0], S[1], hi.x, lo.x);
            split_pair(S[2], S[3], hi.y, lo.y);
            *reinterpret_cast<uint2*>(w + 2 * (size_t)c * step) = hi;
            *reinterpret_cast<uint2*>(w + 2 * (size_t)c * step + (size_t)dv * dp) = lo;
            const float f = c + 1 < chunks ? whole : powf(dec, (float)(nq - c * LC));
            S[0] = fmaf(f, S[0], more[i].x), S[1] = fmaf(f, S[1], more[i].y), S[2] = fmaf(f, S[2], more[i].z), S[3] = fmaf(f, S[3], more[i].w);
        }
    }
    if (vec && n < d) {
        *reinterpret_cast<float4*>(st) = make_float4(S[0], S[1], S[2], S[3]);
    } else {
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (n + i < d) st[i] = S[i];
    }
}

// The outputs of LH tokens of a chunk.  grid: (2 * numbers, heads, tiles of CV values); four warps of 16 tokens each.
// Shared memory: q [LH][dp + 8], then either the start state's parts [2][CV][dp + 8] or k [LH][dp + 8] and v [LH][CV + 8].
constexpr int CV = 64;

__host__ __device__ constexpr size_t lightning_out_smem(int dp) {
    const size_t st = (size_t)2 * CV * (dp + 8), kv = (size_t)LH * (dp + 8) + (size_t)LH * (CV + 8);
    return ((size_t)LH * (dp + 8) + (st > kv ? st : kv)) * 2;
}

__global__ void __launch_bounds__(128, 4) lightning_out_kernel(const __nv_bfloat16* __restrict__ proj, int ld, int H, int d, int dv, int dp,
                                                               const float* __restrict__ decay, const int* __restrict__ cu_q,
                                                               const int* __restrict__ slots, int num_seqs,
                                                               const __nv_bfloat16* __restrict__ starts, float* __restrict__ o, int vec) {
    extern __shared__ __align__(16) __nv_bfloat16 smem[];
    __shared__ float pw[LC + 1];
    const int number = blockIdx.x >> 1, half = blockIdx.x & 1;
    const ChunkAt at = find_chunk(cu_q, num_seqs, number);
    if (at.s < 0 || slots[at.s] < 0) return;
    const int len = min(LC, at.nq - at.c * LC);
    const int i0 = half * LH;                                           // first token of the block within its chunk
    if (i0 >= len) return;
    const int h = blockIdx.y, v0 = blockIdx.z * CV;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row = dp + 8;
    __nv_bfloat16* qs = smem;
    __nv_bfloat16* sh = smem + LH * row;
    __nv_bfloat16* sl = sh + CV * row;
    __nv_bfloat16* ks = smem + LH * row;
    __nv_bfloat16* vs = ks + LH * row;
    const __nv_bfloat16* base = proj + (size_t)(at.q0 + at.c * LC) * ld;
    const __nv_bfloat16* start = starts + 2 * (((size_t)number * H + h) * dv * dp) + (size_t)v0 * dp;
    load_tile(qs, row, base + (size_t)i0 * ld + h * d, ld, LH, dp, len - i0, d, vec);
    load_tile(sh, row, start, dp, CV, dp, dv - v0, dp, 1);
    load_tile(sl, row, start + (size_t)dv * dp, dp, CV, dp, dv - v0, dp, 1);
    const float dec = __ldg(decay + h);
    for (int i = tid; i <= LC; i += 128) pw[i] = powf(dec, (float)i);
    cp_done();
    __syncthreads();
    float acc[CV / 8][4];
#pragma unroll
    for (int i = 0; i < CV / 8; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const __nv_bfloat16* qa = qs + (warp * 16 + (lane & 15)) * row + (lane >> 4) * 8;        // rows of A: this warp's tokens
#pragma unroll 2
    for (int k0 = 0; k0 < dp; k0 += 16) {
        uint32_t a[4];
        ldm4(a, qa + k0);
#pragma unroll
        for (int n = 0; n < CV; n += 16) {
            // (two tiles of eight values: rows n.. and n+8.., channels k0.. and k0+8..)
            const int r = n + (lane & 7) + (lane >= 16 ? 8 : 0), c = k0 + ((lane >> 3) & 1) * 8;
            uint32_t b[4], b2[4];
            ldm4(b, sh + r * row + c);
            ldm4(b2, sl + r * row + c);
            mma16816(acc[n / 8], a, b[0], b[1]);
            mma16816(acc[n / 8 + 1], a, b[2], b[3]);
            mma16816(acc[n / 8], a, b2[0], b2[1]);
            mma16816(acc[n / 8 + 1], a, b2[2], b2[3]);
        }
    }
    const int ia = i0 + warp * 16 + (lane >> 2), ib = ia + 8;           // this lane's tokens within the chunk
    {
        const float fa = pw[min(ia + 1, LC)], fb = pw[min(ib + 1, LC)];
#pragma unroll
        for (int i = 0; i < CV / 8; ++i) acc[i][0] *= fa, acc[i][1] *= fa, acc[i][2] *= fb, acc[i][3] *= fb;
    }
    for (int j0 = 0; j0 <= i0; j0 += LH) {
        __syncthreads();                                                // the state (or the keys in front) has been read
        load_tile(ks, row, base + (size_t)j0 * ld + H * d + h * d, ld, LH, dp, len - j0, d, vec);
        load_tile(vs, CV + 8, base + (size_t)j0 * ld + 2 * H * d + h * dv + v0, ld, LH, CV, len - j0, dv - v0, vec);
        cp_done();
        __syncthreads();
        // the keys that this warp's tokens see: all of an earlier half, else those up to the warp's last token
        const int keys = j0 < i0 ? LH : warp * 16 + 16;
        float sc[LH / 8][4];
#pragma unroll
        for (int i = 0; i < LH / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll 2
        for (int k0 = 0; k0 < dp; k0 += 16) {
            uint32_t a[4];
            ldm4(a, qa + k0);
#pragma unroll
            for (int n = 0; n < LH; n += 16) {
                if (n >= keys) break;
                uint32_t b[4];
                ldm4(b, ks + (n + (lane & 7) + (lane >= 16 ? 8 : 0)) * row + k0 + ((lane >> 3) & 1) * 8);
                mma16816(sc[n / 8], a, b[0], b[1]);
                mma16816(sc[n / 8 + 1], a, b[2], b[3]);
            }
        }
#pragma unroll
        for (int n = 0; n < LH; n += 16) {
            if (n >= keys) break;
            uint32_t ph[4], pl[4];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
                const int j = j0 + n + u * 8 + (lane & 3) * 2;
                float(&x)[4] = sc[n / 8 + u];
                x[0] = j <= ia ? x[0] * pw[ia - j] : 0.f;
                x[1] = j + 1 <= ia ? x[1] * pw[ia - j - 1] : 0.f;
                x[2] = j <= ib ? x[2] * pw[ib - j] : 0.f;
                x[3] = j + 1 <= ib ? x[3] * pw[ib - j - 1] : 0.f;
                split_pair(x[0], x[1], ph[2 * u], pl[2 * u]);
                split_pair(x[2], x[3], ph[2 * u + 1], pl[2 * u + 1]);
            }
#pragma unroll
            for (int v = 0; v < CV; v += 16) {
                uint32_t b[4];
                ldm4t(b, vs + (n + (lane & 7) + ((lane >> 3) & 1) * 8) * (CV + 8) + v + (lane >= 16 ? 8 : 0));
                mma16816(acc[v / 8], ph, b[0], b[1]);
                mma16816(acc[v / 8 + 1], ph, b[2], b[3]);
                mma16816(acc[v / 8], pl, b[0], b[1]);
                mma16816(acc[v / 8 + 1], pl, b[2], b[3]);
            }
        }
    }
    float* out = o + (size_t)(at.q0 + at.c * LC) * H * dv + (size_t)h * dv;
    const bool pairs = (dv & 1) == 0;
#pragma unroll
    for (int i = 0; i < CV / 8; ++i) {
        const int v = v0 + i * 8 + (lane & 3) * 2;
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int t = u ? ib : ia;
            if (t >= len || v >= dv) continue;
            float* p = out + (size_t)t * H * dv + v;
            if (pairs) {
                *reinterpret_cast<float2*>(p) = make_float2(acc[i][2 * u], acc[i][2 * u + 1]);
            } else {
                p[0] = acc[i][2 * u];
                if (v + 1 < dv) p[1] = acc[i][2 * u + 1];
            }
        }
    }
}

// ------------------------------------------------------------------ norm over a row, times a gate
// out[t] = o[t] / sqrt(mean(o[t]^2) + eps) * w * sigmoid(gate[t]); a block per row.
template <typename T>
__global__ void row_norm_gate_kernel(const float* __restrict__ o, const T* __restrict__ gate, int ldg, const float* __restrict__ w,
                                     float eps, T* __restrict__ out, int W, int vec) {
    __shared__ float red[32];
    pdl_launch_dependents();
    pdl_wait();
    const size_t t = blockIdx.x;
    const float* row = o + t * W;
    const T* g = gate + t * ldg;
    T* dst = out + t * W;
    if (vec) {
        // W % 4 == 0 and W <= 16 * threads
        float4 v[4];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            v[i] = c < W ? *reinterpret_cast<const float4*>(row + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
        }
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c >= W) continue;
            const float4 f = *reinterpret_cast<const float4*>(w + c);
            float x[4] = {v[i].x * inv * f.x, v[i].y * inv * f.y, v[i].z * inv * f.z, v[i].w * inv * f.w};
            T y[4];
            T gv[4];
            if (sizeof(T) == 2) *reinterpret_cast<uint2*>(gv) = *reinterpret_cast<const uint2*>(g + c);
            else *reinterpret_cast<uint4*>(gv) = *reinterpret_cast<const uint4*>(g + c);
#pragma unroll
            for (int j = 0; j < 4; ++j) y[j] = from_float<T>(x[j] / (1.0f + expf(-to_float(gv[j]))));
            if (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst + c) = *reinterpret_cast<uint2*>(y);
            else *reinterpret_cast<uint4*>(dst + c) = *reinterpret_cast<uint4*>(y);
        }
        return;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) ss = fmaf(row[c], row[c], ss);
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) dst[c] = from_float<T>(row[c] * inv * __ldg(w + c) / (1.0f + expf(-to_float(g[c]))));
}

template <typename T>
int launch_row_norm_gate(const float* o, const void* gate, int ldg, const float* w, float eps, void* out, long long rows, int W,
                         cudaStream_t stream) {
    const int threads = W >= 4096 ? 512 : W >= 1024 ? 256 : 128;
    const int vec = W % 4 == 0 && ldg % 4 == 0 && W <= threads * 16 &&
                    (((uintptr_t)o | (uintptr_t)w) & 15) == 0 && (((uintptr_t)gate | (uintptr_t)out) & (4 * sizeof(T) - 1)) == 0;
    PL_CUDA(launch_pdl(row_norm_gate_kernel<T>, dim3((unsigned)rows), dim3(threads), 0, stream, o, (const T*)gate, ldg, w, eps, (T*)out, W,
                       vec));
    return 0;
}

template <typename T, int LPC, int NV, int R>
int launch_step(const void* proj, int ld, int H, int d, int dv, const float* decay, float* state, long long state_stride, const int* cu_q,
                const int* slots, int num_seqs, float* o, int vec, cudaStream_t stream) {
    const int cols = 8 * R * (32 / LPC);
    PL_CUDA(launch_pdl(lightning_step_kernel<T, LPC, NV, R>, dim3(num_seqs, H, (dv + cols - 1) / cols), dim3(256), 0, stream, (const T*)proj,
                       ld, H, d, dv, decay, state, state_stride, cu_q, slots, o, vec));
    return 0;
}

template <typename T>
int step_by_size(const void* proj, int ld, int H, int d, int dv, const float* decay, float* state, long long state_stride, const int* cu_q,
                 const int* slots, int num_seqs, float* o, cudaStream_t stream) {
    const int vec = d % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
#define STEP(L, N, R) return launch_step<T, L, N, R>(proj, ld, H, d, dv, decay, state, state_stride, cu_q, slots, num_seqs, o, vec, stream)
    if (d <= 32) STEP(8, 1, 8);
    if (d <= 64) STEP(16, 1, 8);
    if (d <= 128) STEP(32, 1, 8);
    STEP(32, 2, 4);
#undef STEP
}

}  // namespace

// Token by token.
PL_EXPORT int pl_lightning_step(const void* proj, int dtype, int ld, int H, int d, int dv, const float* decay, float* state,
                                long long state_stride, const int* cu_q, const int* slots, int num_seqs, float* o, cudaStream_t stream) {
    if (num_seqs == 0) return 0;
    PL_REQUIRE(H > 0 && H <= 65535 && d > 0 && d <= 256 && dv > 0 && ld >= 2 * H * d + H * dv && state_stride >= (long long)H * d * dv,
               "lightning_step: bad sizes H=%d d=%d dv=%d ld=%d (key size at most 256)", H, d, dv, ld);
    if (dtype == PL_F32) return step_by_size<float>(proj, ld, H, d, dv, decay, state, state_stride, cu_q, slots, num_seqs, o, stream);
    if (dtype == PL_BF16)
        return step_by_size<__nv_bfloat16>(proj, ld, H, d, dv, decay, state, state_stride, cu_q, slots, num_seqs, o, stream);
    return pl_fail("lightning_step: unknown dtype %d", dtype);
}

// In chunks (bfloat16): `numbers` = total_tokens / pl_lightning_chunk() + num_seqs; `buf` holds twice numbers * H * dv * pad16(d)
// floats.  The first 2 * H * d + H * dv columns of proj's `rows` rows are overwritten by their silu.
PL_EXPORT int pl_lightning_chunk() { return LC; }

PL_EXPORT int pl_lightning_chunks(void* proj_, int ld, int rows, int H, int d, int dv, const float* decay, float* buf, int numbers,
                                  float* state, long long state_stride, const int* cu_q, const int* slots, int num_seqs, float* o,
                                  cudaStream_t stream) {
    if (num_seqs == 0 || numbers == 0 || rows == 0) return 0;
    PL_REQUIRE(H > 0 && H <= 65535 && d > 0 && d <= 256 && dv > 0 && dv <= 8192 && ld >= 2 * H * d + H * dv && numbers > 0 && rows > 0 &&
                   state_stride >= (long long)H * d * dv,
               "lightning_chunks: bad sizes H=%d d=%d dv=%d ld=%d (key size at most 256)", H, d, dv, ld);
    __nv_bfloat16* proj = (__nv_bfloat16*)proj_;
    const int dp = (d + 15) / 16 * 16, n = 2 * H * d + H * dv;
    const int vec = ld % 8 == 0 && d % 8 == 0 && dv % 8 == 0 && ((uintptr_t)proj & 15) == 0 && ((uintptr_t)buf & 15) == 0;
    const int vec_state = d % 4 == 0 && state_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    PL_REQUIRE(((uintptr_t)buf & 15) == 0, "lightning_chunks: the scratch is not 16-byte aligned");
    float* add = buf;
    __nv_bfloat16* starts = (__nv_bfloat16*)(buf + (size_t)numbers * H * dv * dp);
    const dim3 grid_s((n / (vec ? 8 : 1) + 255) / 256, rows < 65535 ? rows : 65535);
    PL_CUDA(launch_pdl(lightning_silu_kernel, grid_s, dim3(256), 0, stream, proj, ld, n, rows, vec));
    const dim3 grid_a(numbers, H, (dv + AV - 1) / AV * ((dp + AK - 1) / AK));
    lightning_add_kernel<<<grid_a, 128, 0, stream>>>(proj, ld, H, d, dv, dp, decay, cu_q, slots, num_seqs, add, vec);
    PL_LAUNCHED("lightning_add");
    const dim3 grid_b(num_seqs, H, (dv * dp / 4 + 255) / 256);
    lightning_scan_kernel<<<grid_b, 256, 0, stream>>>(add, starts, H, d, dv, dp, decay, cu_q, slots, state, state_stride, vec_state);
    PL_LAUNCHED("lightning_scan");
    const size_t smem = lightning_out_smem(dp);
    static bool opted[64] = {};
    int dev = 0;
    PL_CUDA(cudaGetDevice(&dev));
    PL_REQUIRE(dev >= 0 && dev < 64, "lightning_chunks: device index %d is out of range", dev);
    if (!opted[dev]) {
        PL_CUDA(cudaFuncSetAttribute(lightning_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)lightning_out_smem(256)));
        opted[dev] = true;
    }
    const dim3 grid_c(2 * numbers, H, (dv + CV - 1) / CV);
    lightning_out_kernel<<<grid_c, 128, smem, stream>>>(proj, ld, H, d, dv, dp, decay, cu_q, slots, num_seqs, starts, o, vec);
    PL_LAUNCHED("lightning_out");
    return 0;
}

PL_EXPORT int pl_row_norm_gate(const float* o, const void* gate, int dtype, int ldg, const float* w, float eps, void* out, long long rows,
                               int W, cudaStream_t stream) {
    if (rows == 0) return 0;
    PL_REQUIRE(rows > 0 && rows < (1ll << 31) && W > 0 && ldg >= W, "row_norm_gate: bad sizes rows=%lld W=%d ldg=%d", rows, W, ldg);
    if (dtype == PL_F32) return launch_row_norm_gate<float>(o, gate, ldg, w, eps, out, rows, W, stream);
    if (dtype == PL_BF16) return launch_row_norm_gate<__nv_bfloat16>(o, gate, ldg, w, eps, out, rows, W, stream);
    return pl_fail("row_norm_gate: unknown dtype %d", dtype);
}
