// Token embedding gather with the additive position table fused in:
// x[t,:] = table[id_t,:] * scale (+ pos_table[pos_t,:]), written as 32-bit, once more to `keep` when a later part of the
// model reads the embedded rows again, and to `act` in the table's dtype when the first layer's products read x itself.
// Same arithmetic as the reference's embedding_kernel (src/kernels/embedding.cu:23-43),
// for any width and either table dtype; row offsets are 64-bit.
#include "common.cuh"

template <typename T>
__global__ void embed_kernel(const int* __restrict__ ids, const int* __restrict__ pos,
                             const T* __restrict__ table, const T* __restrict__ pos_table,
                             float* __restrict__ out, float* __restrict__ keep, T* __restrict__ act, int D, int copies, float scale) {
    const int t = blockIdx.x;
    pdl_launch();               // the first kernel of a step: nothing before it to wait for
    const T* row = table + (size_t)ids[t] * D;
    const T* prow = pos_table ? pos_table + (size_t)pos[t] * D : nullptr;
    float* o = out + (size_t)t * D * copies;
    for (int d = threadIdx.x; d < D; d += blockDim.x) {
        float v = to_f32(row[d]) * scale;
        if (prow) v += to_f32(prow[d]);
        if (keep) keep[(size_t)t * D + d] = v;
        if (act) act[(size_t)t * D + d] = from_f32<T>(v);
        for (int c = 0; c < copies; ++c) o[(size_t)c * D + d] = v;     // a residual of several streams starts as copies
    }
}

MLLM_EXPORT int mllm_embed(const int* ids, const int* pos, const void* table, const void* pos_table,
                           float* out, float* keep, void* act, int T, int D, int copies, float scale, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0 || copies <= 0) return mllm_fail(1, "embed: width %d, %d copies", D, copies);
    int threads = D >= 256 ? 256 : ((D + 31) / 32) * 32;
    if (dtype == MLLM_F32)
        embed_kernel<float><<<T, threads, 0, stream>>>(ids, pos, (const float*)table, (const float*)pos_table, out, keep, (float*)act, D, copies,
                                                    scale);
    else if (dtype == MLLM_BF16)
        embed_kernel<__nv_bfloat16><<<T, threads, 0, stream>>>(ids, pos, (const __nv_bfloat16*)table,
                                                               (const __nv_bfloat16*)pos_table, out, keep, (__nv_bfloat16*)act, D, copies, scale);
    else
        return mllm_fail(1, "embed: unknown dtype code %d", dtype);
    MLLM_CHECK_LAUNCH("embed");
    return 0;
}

// ids[t] < 0 stands for "the token that the last sampling launch wrote to row -ids[t]-1 of
// its output": the step that consumes a token can be queued before the host has read it.
__global__ void resolve_tokens_kernel(int* __restrict__ ids, int T, const int* __restrict__ sampled, int rows) {
    const int t = blockIdx.x * blockDim.x + threadIdx.x;
    if (t >= T) return;
    const int v = ids[t];
    if (v < 0) {
        const int r = -v - 1;
        ids[t] = r < rows ? sampled[r] : 0;
    }
}

MLLM_EXPORT int mllm_resolve_tokens(int* ids, int T, const int* sampled, int rows, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (rows <= 0) return mllm_fail(1, "resolve_tokens: no sampled rows to read from");
    resolve_tokens_kernel<<<(T + 255) / 256, 256, 0, stream>>>(ids, T, sampled, rows);
    MLLM_CHECK_LAUNCH("resolve_tokens");
    return 0;
}

// out[t] = [x hi | x0 hi | x lo | x0 lo] (terms = 2, bfloat16: each value as two bfloat16 terms) or [x | x0] (terms = 1):
// two 32-bit rows side by side as a product reads them.
template <typename T, int TERMS>
__global__ void __launch_bounds__(256)
concat_terms_kernel(const float* x, long long x_stride, const float* x0, long long x0_stride, T* __restrict__ out,
                    long long out_stride, int D) {
    pdl_wait();
    pdl_launch();
    const size_t t = blockIdx.x;
    T* o = out + t * out_stride;
    for (int d = threadIdx.x; d < 2 * D; d += blockDim.x) {
        const float v = d < D ? x[t * x_stride + d] : x0[t * x0_stride + d - D];
        const T hi = from_f32<T>(v);
        o[d] = hi;
        if (TERMS == 2) o[2 * D + d] = from_f32<T>(v - to_f32(hi));
    }
}

MLLM_EXPORT int mllm_concat_terms(const float* x, long long x_stride, const float* x0, long long x0_stride, void* out,
                                  long long out_stride, int T, int D, int terms, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (D <= 0) return mllm_fail(1, "concat_terms: width %d", D);
    if (dtype == MLLM_F32 && terms == 1)
        MLLM_CUDA(mllm_launch(concat_terms_kernel<float, 1>, dim3(T), dim3(256), 0, stream, true, x, x_stride, x0, x0_stride,
                              (float*)out, out_stride, D));
    else if (dtype == MLLM_BF16 && terms == 1)
        MLLM_CUDA(mllm_launch(concat_terms_kernel<__nv_bfloat16, 1>, dim3(T), dim3(256), 0, stream, true, x, x_stride, x0,
                              x0_stride, (__nv_bfloat16*)out, out_stride, D));
    else if (dtype == MLLM_BF16 && terms == 2)
        MLLM_CUDA(mllm_launch(concat_terms_kernel<__nv_bfloat16, 2>, dim3(T), dim3(256), 0, stream, true, x, x_stride, x0,
                              x0_stride, (__nv_bfloat16*)out, out_stride, D));
    else
        return mllm_fail(1, "concat_terms: %d terms of dtype code %d", terms, dtype);
    return 0;
}

// A per-layer input of the token: out[t][c] = gelu_tanh(z[t][c]) * table[ids[t]][off + c], c < d; z 32-bit, table and out in
// the activation dtype.
template <typename T>
__global__ void __launch_bounds__(256)
token_side_gate_kernel(const float* z, long long ldz, const int* __restrict__ ids, const T* __restrict__ table, long long ldt, int off,
                       T* __restrict__ out, long long ldo, int rows, int d) {
    pdl_wait();
    pdl_launch();
    const long long total = (long long)rows * d;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(i / d), c = (int)(i % d);
        out[(size_t)t * ldo + c] = from_f32<T>(gelu_tanh_f(z[(size_t)t * ldz + c]) * to_f32(table[(size_t)ids[t] * ldt + off + c]));
    }
}

MLLM_EXPORT int mllm_token_side_gate(const float* z, long long ldz, const int* ids, const void* table, long long ldt, int off, void* out,
                                     long long ldo, int T, int d, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || off < 0 || off + d > ldt) return mllm_fail(1, "token_side_gate: columns %d to %d of rows of %lld", off, off + d, ldt);
    const long long total = (long long)T * d;
    const int grid = (int)((total + 255) / 256 < 8192 ? (total + 255) / 256 : 8192);
    if (dtype == MLLM_F32)
        MLLM_CUDA(mllm_launch(token_side_gate_kernel<float>, dim3(grid), dim3(256), 0, stream, true, z, ldz, ids, (const float*)table, ldt,
                              off, (float*)out, ldo, T, d));
    else if (dtype == MLLM_BF16)
        MLLM_CUDA(mllm_launch(token_side_gate_kernel<__nv_bfloat16>, dim3(grid), dim3(256), 0, stream, true, z, ldz, ids,
                              (const __nv_bfloat16*)table, ldt, off, (__nv_bfloat16*)out, ldo, T, d));
    else
        return mllm_fail(1, "token_side_gate: unknown dtype code %d", dtype);
    return 0;
}

// Few tokens (decode steps): the gate's product and what token_side_gate makes of it in one launch.  grid (tokens, column
// blocks of 8 * COLS), 8 warps: the token's row of h is staged in shared memory as 32-bit, a warp owns COLS columns and its
// lanes split the sum, with 16-byte loads of the weight rows where they allow it.
template <typename T, int COLS>
__global__ void __launch_bounds__(256)
token_side_mid_kernel(const T* h, long long ldh, const T* __restrict__ W, int D, const int* __restrict__ ids, const T* __restrict__ table,
                      long long ldt, int off, T* __restrict__ out, long long ldo, int d) {
    extern __shared__ float hs[];           // [D]
    constexpr int V = 16 / sizeof(T);
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c0 = (blockIdx.y * 8 + warp) * COLS;
    const T* row = table + (size_t)ids[t] * ldt + off;
    pdl_wait();
    pdl_launch();
    for (int k = threadIdx.x; k < D; k += 256) hs[k] = to_f32(h[(size_t)t * ldh + k]);
    __syncthreads();
    if (c0 >= d) return;
    float acc[COLS];
#pragma unroll
    for (int u = 0; u < COLS; ++u) acc[u] = 0.f;
    if (D % V == 0 && (uintptr_t)W % 16 == 0) {
#pragma unroll 2
        for (int k = lane * V; k < D; k += 32 * V) {
            uint4 w[COLS];
#pragma unroll
            for (int u = 0; u < COLS; ++u) w[u] = *reinterpret_cast<const uint4*>(W + (size_t)min(c0 + u, d - 1) * D + k);
#pragma unroll
            for (int u = 0; u < COLS; ++u) {
                const T* p = reinterpret_cast<const T*>(&w[u]);
#pragma unroll
                for (int e = 0; e < V; ++e) acc[u] = fmaf(hs[k + e], to_f32(p[e]), acc[u]);
            }
        }
    } else {
        for (int k = lane; k < D; k += 32) {
#pragma unroll
            for (int u = 0; u < COLS; ++u) acc[u] = fmaf(hs[k], to_f32(W[(size_t)min(c0 + u, d - 1) * D + k]), acc[u]);
        }
    }
#pragma unroll
    for (int u = 0; u < COLS; ++u) {
        const float v = warp_sum(acc[u]);
        if (lane == 0 && c0 + u < d) out[(size_t)t * ldo + c0 + u] = from_f32<T>(gelu_tanh_f(v) * to_f32(row[c0 + u]));
    }
}

MLLM_EXPORT int mllm_token_side_mid(const void* h, long long ldh, const void* W, int D, const int* ids, const void* table, long long ldt,
                                    int off, void* out, long long ldo, int T, int d, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (d <= 0 || off < 0 || off + d > ldt) return mllm_fail(1, "token_side_mid: columns %d to %d of rows of %lld", off, off + d, ldt);
    if (D <= 0 || (size_t)D * 4 > 48 * 1024) return mllm_fail(1, "token_side_mid: rows of %d", D);
    constexpr int COLS = 2;
    const dim3 grid(T, (d + 8 * COLS - 1) / (8 * COLS));
    if (grid.y > 65535) return mllm_fail(1, "token_side_mid: %d columns", d);
    if (dtype == MLLM_F32)
        MLLM_CUDA(mllm_launch(token_side_mid_kernel<float, COLS>, grid, dim3(256), (size_t)D * 4, stream, true, (const float*)h, ldh,
                              (const float*)W, D, ids, (const float*)table, ldt, off, (float*)out, ldo, d));
    else if (dtype == MLLM_BF16)
        MLLM_CUDA(mllm_launch(token_side_mid_kernel<__nv_bfloat16, COLS>, grid, dim3(256), (size_t)D * 4, stream, true,
                              (const __nv_bfloat16*)h, ldh, (const __nv_bfloat16*)W, D, ids, (const __nv_bfloat16*)table, ldt, off,
                              (__nv_bfloat16*)out, ldo, d));
    else
        return mllm_fail(1, "token_side_mid: unknown dtype code %d", dtype);
    return 0;
}
