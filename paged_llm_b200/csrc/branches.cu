// The sum of a layer's branches with the residual stream.  A branch is a matrix of rows (in either type, with or without a
// bias per column) or the weighted sum of a token's chosen experts' rows that nobody has formed yet.  One kernel, a block
// per row, does
//
//     v = sum of the branches;   x += v (float32 stream, in place);   y = x / sqrt(mean(x^2) + eps) * w   or a copy of x
//
// with everything in float32; without a stream the sum itself is written.
#include "common.cuh"

namespace {

struct Branch {
    const void* rows;       // null (the second one only): no branch
    int bf16;               // type of the rows: 0 float32, 1 bfloat16
    const float* bias;      // [W] or null
    int top;                // > 0: the rows are experts' outputs, `top` of them per token
    const int* place;       // [tokens * top] row of the pair, or null: pair (t, j) is row t * top + j
    const float* weight;    // [tokens * top] or null: the rows carry their weights
    const int* tokens;      // row r stands for this token, or null: token r
};

__device__ __forceinline__ float4 quad(const void* p, int bf16, size_t i) {
    if (!bf16) return *reinterpret_cast<const float4*>(static_cast<const float*>(p) + i);
    const uint2 raw = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + i);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x), b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    return make_float4(__low2float(a), __high2float(a), __low2float(b), __high2float(b));
}

__device__ __forceinline__ float one(const void* p, int bf16, size_t i) {
    return bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]) : static_cast<const float*>(p)[i];
}

__device__ __forceinline__ void put_quad(void* p, int bf16, size_t i, float4 v) {
    if (!bf16) {
        *reinterpret_cast<float4*>(static_cast<float*>(p) + i) = v;
        return;
    }
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + i) = raw;
}

constexpr int QUADS = 4;        // quads of a row per thread in the vector form

// v[i] += the branch at this thread's quads of row r.  Experts' rows come four at a time, all quads of the four at once.
template <bool BF16>
__device__ __forceinline__ void add_branch(const Branch& b, int r, int W, float4 (&v)[QUADS]) {
    if (b.top > 0) {
        const size_t first = (size_t)(b.tokens != nullptr ? b.tokens[r] : r) * b.top;
        for (int j0 = 0; j0 < b.top; j0 += 4) {
            long long row[4];
            float w[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const bool in = j0 + j < b.top;
                row[j] = !in ? -1 : b.place != nullptr ? (long long)b.place[first + j0 + j] : (long long)(first + j0 + j);
                w[j] = in && b.weight != nullptr ? b.weight[first + j0 + j] : 1.f;
            }
#pragma unroll
            for (int i = 0; i < QUADS; ++i) {
                const int c = (threadIdx.x + i * blockDim.x) * 4;
                if (c >= W) break;
                float4 e[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) e[j] = row[j] >= 0 ? quad(b.rows, BF16, (size_t)row[j] * W + c) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    v[i].x = fmaf(w[j], e[j].x, v[i].x), v[i].y = fmaf(w[j], e[j].y, v[i].y), v[i].z = fmaf(w[j], e[j].z, v[i].z),
                    v[i].w = fmaf(w[j], e[j].w, v[i].w);
            }
        }
        return;
    }
#pragma unroll
    for (int i = 0; i < QUADS; ++i) {
        const int c = (threadIdx.x + i * blockDim.x) * 4;
        if (c >= W) break;
        float4 s = quad(b.rows, BF16, (size_t)r * W + c);
        if (b.bias != nullptr) {
            const float4 t = *reinterpret_cast<const float4*>(b.bias + c);
            s = make_float4(s.x + t.x, s.y + t.y, s.z + t.z, s.w + t.w);
        }
        v[i] = make_float4(v[i].x + s.x, v[i].y + s.y, v[i].z + s.z, v[i].w + s.w);
    }
}

__device__ __forceinline__ float branch_one(const Branch& b, int r, int c, int W) {
    float s = 0.f;
    if (b.top > 0) {
        const size_t first = (size_t)(b.tokens != nullptr ? b.tokens[r] : r) * b.top;
        for (int j = 0; j < b.top; ++j) {
            const long long row = b.place != nullptr ? b.place[first + j] : (long long)(first + j);
            if (row >= 0) s = fmaf(b.weight != nullptr ? b.weight[first + j] : 1.f, one(b.rows, b.bf16, (size_t)row * W + c), s);
        }
    } else {
        s = one(b.rows, b.bf16, (size_t)r * W + c);
    }
    return b.bias != nullptr ? s + __ldg(b.bias + c) : s;
}

__global__ void branch_norm_kernel(float* __restrict__ x, Branch a, Branch b, const void* __restrict__ w, int w_bf16, void* __restrict__ y,
                                   int y_bf16, int W, float eps, int vec) {
    __shared__ float red[32];
    pdl_launch_dependents();
    const int r = blockIdx.x;
    const size_t base = (size_t)r * W;
    pdl_wait();
    if (vec) {
        // W % 4 == 0 and W <= 4 * QUADS * threads: the row lives in registers
        float4 v[QUADS];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < QUADS; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            v[i] = x != nullptr && c < W ? *reinterpret_cast<const float4*>(x + base + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        if (a.bf16) add_branch<true>(a, r, W, v); else add_branch<false>(a, r, W, v);
        if (b.rows != nullptr) {
            if (b.bf16) add_branch<true>(b, r, W, v); else add_branch<false>(b, r, W, v);
        }
#pragma unroll
        for (int i = 0; i < QUADS; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < W) {
                if (x != nullptr) *reinterpret_cast<float4*>(x + base + c) = v[i];
                if (w == nullptr && y != nullptr) put_quad(y, y_bf16, base + c, v[i]);
                ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
            }
        }
        if (w == nullptr) return;
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
#pragma unroll
        for (int i = 0; i < QUADS; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * 4;
            if (c < W) {
                const float4 g = quad(w, w_bf16, c);
                put_quad(y, y_bf16, base + c, make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w));
            }
        }
        return;
    }
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float v = x != nullptr ? x[base + c] : 0.f;
        v += branch_one(a, r, c, W);
        if (b.rows != nullptr) v += branch_one(b, r, c, W);
        if (x != nullptr) x[base + c] = v;
        if (w == nullptr && y != nullptr) {
            if (y_bf16) static_cast<__nv_bfloat16*>(y)[base + c] = __float2bfloat16_rn(v);
            else static_cast<float*>(y)[base + c] = v;
        }
        ss = fmaf(v, v, ss);
    }
    if (w == nullptr) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)W + eps);
    for (int c = threadIdx.x; c < W; c += blockDim.x) {         // (a thread reads back what it wrote itself)
        const float v = x[base + c] * inv * one(w, w_bf16, c);
        if (y_bf16) static_cast<__nv_bfloat16*>(y)[base + c] = __float2bfloat16_rn(v);
        else static_cast<float*>(y)[base + c] = v;
    }
}

}  // namespace

// Branch a (and b, or b_rows null): rows, dtype, bias, and for experts' rows top > 0, place, weight, tokens.  x null: y gets
// the sum of the branches; w null: y (may be null) gets a copy of x; else its norm.
PL_EXPORT int pl_branch_norm(float* x, const void* a_rows, int a_dtype, const float* a_bias, int a_top, const int* a_place,
                             const float* a_weight, const int* a_tokens, const void* b_rows, int b_dtype, const float* b_bias, int b_top,
                             const int* b_place, const float* b_weight, const int* b_tokens, const void* w, int w_dtype, void* y,
                             int y_dtype, long long rows, int W, float eps, cudaStream_t stream) {
    if (rows == 0) return 0;
    PL_REQUIRE(rows > 0 && rows < (1ll << 31) && W > 0, "branch_norm: bad sizes rows=%lld W=%d", rows, W);
    PL_REQUIRE(a_rows != nullptr && (x != nullptr || (y != nullptr && w == nullptr)) && (w == nullptr || y != nullptr),
               "branch_norm: nothing to add, or nowhere to write");
    PL_REQUIRE((a_dtype | b_dtype | w_dtype | y_dtype) <= 1 && a_top >= 0 && b_top >= 0, "branch_norm: unknown dtype");
    const Branch a = {a_rows, a_dtype, a_bias, a_top, a_place, a_weight, a_tokens};
    const Branch b = {b_rows, b_dtype, b_bias, b_top, b_place, b_weight, b_tokens};
    const int threads = W >= 4096 ? 512 : W >= 1024 ? 256 : 128;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)a_rows | (uintptr_t)a_bias | (uintptr_t)b_rows | (uintptr_t)b_bias | (uintptr_t)w | (uintptr_t)y;
    const int vec = W % 4 == 0 && W <= threads * 4 * QUADS && (all & 15) == 0;
    PL_CUDA(launch_pdl(branch_norm_kernel, dim3((unsigned)rows), dim3(threads), 0, stream, x, a, b, w, w_dtype, y, y_dtype, W, eps, vec));
    return 0;
}
