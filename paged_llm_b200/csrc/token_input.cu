// What a token brings to the stream beside its embedding row, and small pieces around it:
//
//  * the embedding's rows times a factor plus a sinusoidal vector of the position;
//  * the residual sum with a copy of the new stream in the activations' type (the operand of a product that reads the
//    stream itself, without a norm);
//  * the gate of a per-layer token vector: gelu_tanh(z) * table[id, part of the layer];
//  * a cap on logits.
//
// The stream, angles, activations and sums are float32 whatever the activations' type is.
#include "common.cuh"

// ------------------------------------------------------------------ embedding + sinusoidal position
// out[t, 2i] = table[id, 2i] * scale + sin(2 pi p turns[i]), out[t, 2i+1] the same with cos; p the token's position.
// `turns` (turns of the circle per position) and the reduction to one turn are double, so that the phase is exact far out.
__device__ __forceinline__ float4 quad(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 quad(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}

__device__ __forceinline__ void sinusoid(double turns, double p, float& sn, float& cs) {
    const double ph = p * turns;
    sincospif(2.0f * (float)(ph - rint(ph)), &sn, &cs);
}

// grid: (blocks of a row, tokens).  vec: four elements per thread (H % 4 == 0, 16-byte aligned rows).
template <typename TW>
__global__ void __launch_bounds__(128) embedding_sinusoid_kernel(const TW* __restrict__ table, const int* __restrict__ ids,
                                                                 const int* __restrict__ positions, const double* __restrict__ turns,
                                                                 float* __restrict__ out, int H, int V, float scale, int vec) {
    pdl_launch_dependents();
    const int first = blockIdx.x * blockDim.x + threadIdx.x, stride = gridDim.x * blockDim.x;
    const int t = blockIdx.y;
    pdl_wait();
    const int id = ids[t];
    const double p = (double)positions[t];
    const bool valid = id >= 0 && id < V;
    const TW* row = table + (size_t)(valid ? id : 0) * H;
    float* o = out + (size_t)t * H;
    if (vec) {
        for (int c = first * 4; c < H; c += stride * 4) {
            const double2 tu = *reinterpret_cast<const double2*>(turns + c / 2);
            float4 v = quad(row + c), e;
            if (!valid) v = make_float4(0.f, 0.f, 0.f, 0.f);
            sinusoid(tu.x, p, e.x, e.y);
            sinusoid(tu.y, p, e.z, e.w);
            *reinterpret_cast<float4*>(o + c) = make_float4(fmaf(v.x, scale, e.x), fmaf(v.y, scale, e.y), fmaf(v.z, scale, e.z), fmaf(v.w, scale, e.w));
        }
        return;
    }
    for (int i = first; 2 * i < H; i += stride) {
        float sn, cs;
        sinusoid(turns[i], p, sn, cs);
        o[2 * i] = (valid ? to_float(row[2 * i]) * scale : 0.f) + sn;
        if (2 * i + 1 < H) o[2 * i + 1] = (valid ? to_float(row[2 * i + 1]) * scale : 0.f) + cs;
    }
}

PL_EXPORT int pl_embedding_sinusoid(const void* table, int table_dtype, const int* ids, const int* positions, const double* turns,
                                    float* out, int T, int H, int V, float scale, cudaStream_t stream) {
    if (T == 0) return 0;
    PL_REQUIRE(T > 0 && H > 0 && V > 0, "embedding_sinusoid: bad sizes T=%d H=%d V=%d", T, H, V);
    PL_REQUIRE(T <= 65535 * 32, "embedding_sinusoid: %d tokens", T);
    const int vec = H % 4 == 0 && (((uintptr_t)table | (uintptr_t)out | (uintptr_t)turns) & 15) == 0;
    const int bx = ((vec ? H / 4 : (H + 1) / 2) + 127) / 128;
    for (int t0 = 0; t0 < T; t0 += 65535) {                       // (the y extent of a grid)
        const int n = T - t0 < 65535 ? T - t0 : 65535;
        if (table_dtype == PL_F32)
            PL_CUDA(launch_pdl(embedding_sinusoid_kernel<float>, dim3(bx, n), dim3(128), 0, stream, (const float*)table, ids + t0,
                               positions + t0, turns, out + (size_t)t0 * H, H, V, scale, vec));
        else if (table_dtype == PL_BF16)
            PL_CUDA(launch_pdl(embedding_sinusoid_kernel<__nv_bfloat16>, dim3(bx, n), dim3(128), 0, stream, (const __nv_bfloat16*)table,
                               ids + t0, positions + t0, turns, out + (size_t)t0 * H, H, V, scale, vec));
        else
            return pl_fail("embedding_sinusoid: unknown dtype %d", table_dtype);
    }
    return 0;
}

// ------------------------------------------------------------------ residual sum + a copy in the activations' type
template <typename TB>
__global__ void __launch_bounds__(256) add_copy_kernel(float* __restrict__ x, const TB* __restrict__ branch,
                                                       __nv_bfloat16* __restrict__ copy, long long n, int vec) {
    pdl_launch_dependents();
    pdl_wait();
    const long long stride = (long long)gridDim.x * blockDim.x;
    if (vec) {
        for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * 4; i < n; i += stride * 4) {
            float4 v = *reinterpret_cast<const float4*>(x + i);
            if (branch != nullptr) {
                const float4 b = quad(branch + i);
                v = make_float4(v.x + b.x, v.y + b.y, v.z + b.z, v.w + b.w);
                *reinterpret_cast<float4*>(x + i) = v;
            }
            __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
            uint2 raw;
            raw.x = *reinterpret_cast<uint32_t*>(&lo);
            raw.y = *reinterpret_cast<uint32_t*>(&hi);
            *reinterpret_cast<uint2*>(copy + i) = raw;
        }
        return;
    }
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) {
        float v = x[i];
        if (branch != nullptr) {
            v += to_float(branch[i]);
            x[i] = v;
        }
        copy[i] = __float2bfloat16_rn(v);
    }
}

// x += branch (float32 or bfloat16, may be null), copy = bfloat16(x).
PL_EXPORT int pl_add_copy(float* x, const void* branch, int branch_dtype, void* copy, long long n, cudaStream_t stream) {
    if (n == 0) return 0;
    PL_REQUIRE(n > 0 && copy != nullptr, "add_copy: bad arguments");
    const int vec = n % 4 == 0 && (((uintptr_t)x | (uintptr_t)branch | (uintptr_t)copy) & 15) == 0;
    const long long units = vec ? n / 4 : n, want = (units + 255) / 256;
    const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
    if (branch == nullptr || branch_dtype == PL_F32)
        PL_CUDA(launch_pdl(add_copy_kernel<float>, dim3(blocks), dim3(256), 0, stream, x, (const float*)branch, (__nv_bfloat16*)copy, n, vec));
    else if (branch_dtype == PL_BF16)
        PL_CUDA(launch_pdl(add_copy_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, x, (const __nv_bfloat16*)branch,
                           (__nv_bfloat16*)copy, n, vec));
    else
        return pl_fail("add_copy: unknown dtype %d", branch_dtype);
    return 0;
}

// ------------------------------------------------------------------ gate on a per-layer token vector
// out[t, j] = gelu_tanh(z[t, j]) * table[ids[t], col0 + j] for j < dim, 0 for dim <= j < n (columns that pad a product).
template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(const T* __restrict__ z, const T* __restrict__ table, int ldt, int col0, int dim,
                                                         const int* __restrict__ ids, int V, T* __restrict__ out, int n, long long total) {
    pdl_launch_dependents();
    pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long t = i / n;
        const int j = (int)(i - t * n), id = ids[t];
        const float e = j < dim && id >= 0 && id < V ? to_float(table[(size_t)id * ldt + col0 + j]) : 0.f;
        out[i] = from_float<T>(gelu_tanh_f(to_float(z[i])) * e);
    }
}

PL_EXPORT int pl_token_gate(const void* z, int dtype, const void* table, int ldt, int col0, int dim, const int* ids, int V, void* out,
                            int rows, int n, cudaStream_t stream) {
    if (rows == 0) return 0;
    PL_REQUIRE(rows > 0 && dim > 0 && dim <= n && V > 0 && col0 >= 0 && col0 + dim <= ldt, "token_gate: columns %d..%d of %d", col0,
               col0 + dim, ldt);
    const long long total = (long long)rows * n, want = (total + 255) / 256;
    const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
    if (dtype == PL_F32)
        PL_CUDA(launch_pdl(token_gate_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)z, (const float*)table, ldt, col0, dim,
                           ids, V, (float*)out, n, total));
    else if (dtype == PL_BF16)
        PL_CUDA(launch_pdl(token_gate_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)z,
                           (const __nv_bfloat16*)table, ldt, col0, dim, ids, V, (__nv_bfloat16*)out, n, total));
    else
        return pl_fail("token_gate: unknown dtype %d", dtype);
    return 0;
}

// ------------------------------------------------------------------ elementwise activations of a product's columns
// out[r, c] = f(in[r, col0 + c]), c < n; f: 3 the square of relu, 4 tanh.
template <typename T>
__global__ void __launch_bounds__(256) act_columns_kernel(const T* __restrict__ in, int ld, int col0, T* __restrict__ out, int n, int act,
                                                          long long total) {
    pdl_launch_dependents();
    pdl_wait();
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const long long r = i / n;
        const float v = to_float(in[r * ld + col0 + (i - r * n)]);
        out[i] = from_float<T>(act == 3 ? relu2_f(v) : tanhf(v));
    }
}

PL_EXPORT int pl_act_columns(const void* in, int dtype, int ld, int col0, void* out, int rows, int n, int act, cudaStream_t stream) {
    if (rows == 0) return 0;
    PL_REQUIRE(rows > 0 && n > 0 && col0 >= 0 && col0 + n <= ld, "act_columns: columns %d..%d of %d", col0, col0 + n, ld);
    PL_REQUIRE(act == 3 || act == 4, "act_columns: unknown activation %d", act);
    const long long total = (long long)rows * n, want = (total + 255) / 256;
    const unsigned blocks = (unsigned)(want < 148 * 16 ? want : 148 * 16);
    if (dtype == PL_F32)
        PL_CUDA(launch_pdl(act_columns_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)in, ld, col0, (float*)out, n, act,
                           total));
    else if (dtype == PL_BF16)
        PL_CUDA(launch_pdl(act_columns_kernel<__nv_bfloat16>, dim3(blocks), dim3(256), 0, stream, (const __nv_bfloat16*)in, ld, col0,
                           (__nv_bfloat16*)out, n, act, total));
    else
        return pl_fail("act_columns: unknown dtype %d", dtype);
    return 0;
}

// ------------------------------------------------------------------ cap on logits
// x <- cap * tanh(x / cap) in place.
__global__ void __launch_bounds__(256) softcap_kernel(float* __restrict__ x, long long n, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const float inv = 1.0f / cap;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long long)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv);
}

PL_EXPORT int pl_softcap(float* x, long long n, float cap, cudaStream_t stream) {
    if (n == 0) return 0;
    PL_REQUIRE(n > 0 && cap > 0.f, "softcap: n=%lld cap=%g", n, (double)cap);
    const long long want = (n + 255) / 256;
    PL_CUDA(launch_pdl(softcap_kernel, dim3((unsigned)(want < 148 * 16 ? want : 148 * 16)), dim3(256), 0, stream, x, n, cap));
    return 0;
}
