// The selective scan with a state vector per channel (Mamba's first form).  A channel with rates a in R^N (negative), a skip
// factor d and a state s in R^N (at first zeros) takes, token after token, an input x, a gate z, a raw step size and the two
// vectors B, C that all channels of the token share:
//   h = softplus(raw + bias)        s <- e^(h a) * s + h x B   (entry by entry)        out = out_scale * (s . C + d x) * silu(z)
// x (the convolution's output), B, C and z come in the activation dtype; dt, the decays, the state and the sums are 32-bit.
//
// `scan` (prompt portions): a CTA takes 128 / L channels of one request.  128 threads walk: L lanes share a channel and keep R
// consecutive state entries each in registers throughout; the decays do not depend on the state, so only one fused
// multiply-add per entry is sequential, and four tokens' sums over the lanes meet together.  128 more threads bring the
// inputs, three chunks of 16 (8) tokens ahead and through registers, take softplus once per (token, channel) on the way to
// shared memory, and gate and store the chunk that was walked last: one barrier per chunk.  `step` (single tokens): the step
// size's projection, softplus, update, output and gate in one launch; S, A and the projection's weights are read before the
// kernel waits for its predecessor.
// Every state entry is a recurrence of its own and both kernels do the same operations per token, so the state after some
// tokens is the same bits however they were cut into portions (single tokens make dt in another summation order).
#include "common.cuh"

namespace {

constexpr int THREADS = 128;
constexpr float LOG2E = 1.4426950408889634f;

struct SelArgs {
    const float* A;                 // [C][N] the channels' rates
    const float* skip;              // [C]
    const float* bias;              // [C] of the step sizes
    float* state;                   // [slots][stride]: S [C][N] at the row's start
    long long stride;
    const int* cu_q;
    const int* slots;
    int C, N, write_state;
    float out_scale;
};

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// silu for a result that is rounded to T: with bfloat16 the fast exponential and division (about 1e-6) are far below that rounding
template <typename T> __device__ __forceinline__ float silu_out(float v) {
    if constexpr (sizeof(T) == 4) return silu_f(v);
    return __fdividef(v, 1.0f + __expf(-v));
}

// exp(dt * a): on the bfloat16 path the rates are kept in units of ln 2 and the exponential is one instruction
template <typename T> __device__ __forceinline__ float rate_unit() { return sizeof(T) == 4 ? 1.0f : LOG2E; }
template <typename T> __device__ __forceinline__ float decay_of(float dt, float a) {
    if constexpr (sizeof(T) == 4) return expf(dt * a);
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(dt * a));
    return y;
}

template <typename T, int R>
__device__ __forceinline__ float advance(float* s, const float* ar, float dt, float dx, const float* b, const float* c) {
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < R; i += 4) {
        const float4 bv = *reinterpret_cast<const float4*>(b + i), cv = *reinterpret_cast<const float4*>(c + i);
        s[i] = fmaf(decay_of<T>(dt, ar[i]), s[i], dx * bv.x);
        s[i + 1] = fmaf(decay_of<T>(dt, ar[i + 1]), s[i + 1], dx * bv.y);
        s[i + 2] = fmaf(decay_of<T>(dt, ar[i + 2]), s[i + 2], dx * bv.z);
        s[i + 3] = fmaf(decay_of<T>(dt, ar[i + 3]), s[i + 3], dx * bv.w);
        acc += (s[i] * cv.x + s[i + 1] * cv.y) + (s[i + 2] * cv.z + s[i + 3] * cv.w);
    }
    return acc;
}

template <int L>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// grid (channel blocks, requests); the first 128 threads walk the tokens, the other 128 bring and carry away (see the top).
// x [T][ldx], raw step sizes dt [T][lddt] (32-bit, bias not yet added), bc [T][ldbc] with B at b_off and C at c_off,
// z [T][ldz], out [T][ldo].
template <typename T, int L, int R>
__global__ void __launch_bounds__(2 * THREADS)
selective_scan_kernel(const T* x, long long ldx, const float* dt, long long lddt, const T* bc, long long ldbc, int b_off,
                      int c_off, const T* z, long long ldz, T* __restrict__ out, long long ldo, SelArgs a) {
    constexpr int CPB = THREADS / L, NR = L * R, CH = (NR > 128 || L == 1) ? 8 : 16;
    constexpr int NB = (CH * NR + THREADS - 1) / THREADS, NX = (CH * CPB + THREADS - 1) / THREADS;
    __shared__ __align__(16) float Bs[2][CH * NR], Cs[2][CH * NR];
    __shared__ float2 dx[2][CH * CPB];          // (dt, dt * x)
    __shared__ float ys[2][CH * CPB];
    const bool walker = threadIdx.x < THREADS;
    const int tid = threadIdx.x % THREADS, seq = blockIdx.y, base = blockIdx.x * CPB;
    const int ch = tid / L, lane = tid % L, c = base + ch;
    const bool live = walker && c < a.C;
    float ar[R], s[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = lane * R + i;
        ar[i] = live && r < a.N ? a.A[(size_t)c * a.N + r] * rate_unit<T>() : 0.f;
    }
    pdl_wait();
    pdl_launch();
    const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
    if (n <= 0) return;
    const int chunks = (n + CH - 1) / CH;
    float* S = a.state + (size_t)a.slots[seq] * a.stride + (size_t)c * a.N;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = lane * R + i;
        s[i] = live && r < a.N ? S[r] : 0.f;
    }
    // what the second half holds between iterations: the raw inputs of the next two chunks to be walked, and z and x of the
    // two whose results are still to be stored; a load has two iterations to arrive
    struct In { T b[NB], c[NB], x[NX]; float d[NX]; } in0, in1;
    struct Out { T z[NX], x[NX]; } out0, out1;
    const int mine = base + tid % CPB;          // this thread's channel when it brings or carries away
    const float bias = mine < a.C ? a.bias[mine] : 0.f, skip = mine < a.C ? a.skip[mine] : 0.f;
    // Row numbers and columns are held inside the tensors instead of asking before every load: what a token beyond the portion
    // or a channel beyond the last brings is never used.  Token tid / CPB + u * L of a chunk, one channel throughout.
    const int mine_in = min(mine, a.C - 1), first = tid / CPB;
    const char* px = reinterpret_cast<const char*>(x + (size_t)t0 * ldx + mine_in);
    const char* pz = reinterpret_cast<const char*>(z + (size_t)t0 * ldz + mine_in);
    const char* pd = reinterpret_cast<const char*>(dt + (size_t)t0 * lddt + mine_in);
    const char* pb = reinterpret_cast<const char*>(bc + (size_t)t0 * ldbc + b_off);
    const ptrdiff_t to_c = (ptrdiff_t)(c_off - b_off) * (ptrdiff_t)sizeof(T);
    const unsigned sx = (unsigned)(ldx * sizeof(T)), sz = (unsigned)(ldz * sizeof(T)), sd = (unsigned)(lddt * 4), sb = (unsigned)(ldbc * sizeof(T));
    auto at = [](const char* p, unsigned row, unsigned stride) { return p + (unsigned long long)row * stride; };
    auto fetch = [&](int k, In& r) {
        if (k >= chunks) return;
#pragma unroll
        for (int u = 0; u < NB; ++u) {
            const int i = tid + u * THREADS, e = i % NR;
            const char* row = at(pb, min(k * CH + i / NR, n - 1), sb) + min(e, a.N - 1) * (int)sizeof(T);
            r.b[u] = *reinterpret_cast<const T*>(row);
            r.c[u] = *reinterpret_cast<const T*>(row + to_c);
        }
#pragma unroll
        for (int u = 0; u < NX; ++u) {
            const unsigned t = min(k * CH + first + u * L, n - 1);
            r.x[u] = *reinterpret_cast<const T*>(at(px, t, sx));
            r.d[u] = *reinterpret_cast<const float*>(at(pd, t, sd));
        }
    };
    auto put = [&](int k, const In& r) {
        if (k >= chunks) return;
        const int buf = k & 1;
#pragma unroll
        for (int u = 0; u < NB; ++u) {
            const int i = tid + u * THREADS;
            const bool ok = i % NR < a.N;               // entries beyond the state stay zero
            if (i < CH * NR) { Bs[buf][i] = ok ? to_f32(r.b[u]) : 0.f; Cs[buf][i] = ok ? to_f32(r.c[u]) : 0.f; }
        }
#pragma unroll
        for (int u = 0; u < NX; ++u) {
            const int i = tid + u * THREADS;
            const float d = softplus_f(r.d[u] + bias);
            if (i < CH * CPB) dx[buf][i] = make_float2(d, d * to_f32(r.x[u]));
        }
    };
    auto fetch_out = [&](int k, Out& o) {
        if (k >= chunks) return;
#pragma unroll
        for (int u = 0; u < NX; ++u) {
            const unsigned t = min(k * CH + first + u * L, n - 1);
            o.z[u] = *reinterpret_cast<const T*>(at(pz, t, sz));
            o.x[u] = *reinterpret_cast<const T*>(at(px, t, sx));
        }
    };
    char* po = reinterpret_cast<char*>(out + (size_t)t0 * ldo + mine_in);
    const unsigned so = (unsigned)(ldo * sizeof(T));
    auto put_out = [&](int k, const Out& o) {
        if (k < 0 || mine >= a.C) return;
#pragma unroll
        for (int u = 0; u < NX; ++u) {
            const int i = tid + u * THREADS, t = k * CH + first + u * L;
            if (i < CH * CPB && t < n)
                *reinterpret_cast<T*>(po + (unsigned long long)(unsigned)t * so) =
                    from_f32<T>(fmaf(skip, to_f32(o.x[u]), ys[k & 1][i]) * silu_out<T>(to_f32(o.z[u])) * a.out_scale);
        }
    };
    auto bring = [&](int k, In& next, Out& done) {          // next: chunk k + 1; done: chunk k - 1
        put(k + 1, next);
        put_out(k - 1, done);
        fetch(k + 3, next);
        fetch_out(k + 1, done);
    };
    auto walk = [&](int k) {
        const int nc = min(CH, n - k * CH);
        const float2* dk = dx[k & 1] + ch;
        const float *bk = Bs[k & 1] + lane * R, *ck = Cs[k & 1] + lane * R;
        float* yk = ys[k & 1] + ch;
        auto token = [&](int tt) {
            const float2 d = dk[tt * CPB];
            return advance<T, R>(s, ar, d.x, d.y, bk + tt * NR, ck + tt * NR);
        };
        if (L >= 4 && nc == CH) {
            // four tokens together: their sums over the L lanes meet by halving, and a lane ends with one token's.  Nothing is
            // stored before the whole chunk has been walked, so that later tokens' loads are not held up.
            const bool up1 = lane & (L / 2), up2 = lane & (L / 4);
            float w[CH / 4];
#pragma unroll
            for (int q = 0; q < CH / 4; ++q) {
                const float v0 = token(4 * q), v1 = token(4 * q + 1), v2 = token(4 * q + 2), v3 = token(4 * q + 3);
                const float h0 = (up1 ? v2 : v0) + __shfl_xor_sync(0xffffffffu, up1 ? v0 : v2, L / 2);
                const float h1 = (up1 ? v3 : v1) + __shfl_xor_sync(0xffffffffu, up1 ? v1 : v3, L / 2);
                w[q] = (up2 ? h1 : h0) + __shfl_xor_sync(0xffffffffu, up2 ? h0 : h1, L / 4);
#pragma unroll
                for (int o = L / 8; o > 0; o >>= 1) w[q] += __shfl_xor_sync(0xffffffffu, w[q], o);
            }
            if (L == 4 || (lane & (L / 4 - 1)) == 0) {
                const int at = (up1 ? 2 : 0) + (up2 ? 1 : 0);
#pragma unroll
                for (int q = 0; q < CH / 4; ++q) yk[(4 * q + at) * CPB] = w[q];
            }
            return;
        }
        for (int tt = 0; tt < nc; ++tt) {
            const float w = lanes_sum<L>(token(tt));
            if (lane == 0) yk[tt * CPB] = w;
        }
    };
    if (!walker) {
        fetch(0, in0);
        fetch(1, in1);
        put(0, in0);
        fetch(2, in0);
        fetch_out(0, out0);
    }
    for (int k = 0; k <= chunks; ++k) {
        __syncthreads();                        // chunk k is in; what was walked last is complete
        if (walker) {
            if (k < chunks) walk(k);
        } else if (k & 1) {                     // chunk k + 1 came into in0, chunk k - 1's outputs wait for out0
            bring(k, in0, out0);
        } else {
            bring(k, in1, out1);
        }
    }
    if (a.write_state && live) {
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (lane * R + i < a.N) S[lane * R + i] = s[i];
    }
}

// Single tokens: grid (channel blocks, requests).  low [T][ldlow]: the step sizes' low-rank columns (rank), B at b_off, C at
// c_off; W [C][rank8], rank8 the rank rounded up to 8, zeros beyond the rank.
template <typename T, int L, int R>
__global__ void __launch_bounds__(THREADS)
selective_step_kernel(const T* x, long long ldx, const T* low, long long ldlow, int rank, int b_off, int c_off,
                      const T* __restrict__ W, const T* z, long long ldz, T* __restrict__ out, long long ldo, SelArgs a) {
    constexpr int CPB = THREADS / L, NR = L * R, V = 16 / sizeof(T);
    extern __shared__ __align__(16) float lows[];               // [rank8]
    __shared__ __align__(16) float Bs[NR], Cs[NR];
    const int tid = threadIdx.x, seq = blockIdx.y;
    const int ch = tid / L, lane = tid % L, c = blockIdx.x * CPB + ch;
    const int rank8 = (rank + 7) / 8 * 8;
    const bool live = c < a.C;
    const int t = a.cu_q[seq];
    float* S = a.state + (size_t)a.slots[seq] * a.stride + (size_t)c * a.N;
    float ar[R], s[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int r = lane * R + i;
        const bool ok = live && r < a.N;
        ar[i] = ok ? a.A[(size_t)c * a.N + r] * rate_unit<T>() : 0.f;
        s[i] = ok ? S[r] : 0.f;
    }
    const T* wr = W + (size_t)(live ? c : 0) * rank8;
    uint4 first = make_uint4(0u, 0u, 0u, 0u);
    if (lane * V < rank8) first = *reinterpret_cast<const uint4*>(wr + lane * V);
    const float skip = live ? a.skip[c] : 0.f, bias = live ? a.bias[c] : 0.f;
    pdl_wait();
    pdl_launch();
    const T* lr = low + (size_t)t * ldlow;
    for (int r = tid; r < rank8; r += THREADS) lows[r] = r < rank ? to_f32(lr[r]) : 0.f;
    for (int r = tid; r < NR; r += THREADS) {
        Bs[r] = r < a.N ? to_f32(lr[b_off + r]) : 0.f;
        Cs[r] = r < a.N ? to_f32(lr[c_off + r]) : 0.f;
    }
    const float xv = live ? to_f32(x[(size_t)t * ldx + c]) : 0.f;
    const float zv = live && lane == 0 ? to_f32(z[(size_t)t * ldz + c]) : 0.f;
    __syncthreads();
    float acc = 0.f;
    for (int r = lane * V; r < rank8; r += L * V) {
        const uint4 w4 = r == lane * V ? first : *reinterpret_cast<const uint4*>(wr + r);
        const T* w = reinterpret_cast<const T*>(&w4);
#pragma unroll
        for (int e = 0; e < V; ++e) acc = fmaf(to_f32(w[e]), lows[r + e], acc);
    }
    const float d = softplus_f(lanes_sum<L>(acc) + bias);
    const float y = lanes_sum<L>(advance<T, R>(s, ar, d, d * xv, Bs + lane * R, Cs + lane * R));
    if (!live) return;
    if (lane == 0) out[(size_t)t * ldo + c] = from_f32<T>(fmaf(skip, xv, y) * silu_out<T>(zv) * a.out_scale);
    if (a.write_state) {
#pragma unroll
        for (int i = 0; i < R; ++i)
            if (lane * R + i < a.N) S[lane * R + i] = s[i];
    }
}

int check(const char* what, const SelArgs& a, int S) {
    if (a.C <= 0 || a.N <= 0 || a.N > 256) return mllm_fail(1, "%s: %d channels with states of %d entries (at most 256)", what, a.C, a.N);
    if (a.C > (1 << 26)) return mllm_fail(1, "%s: %d channels", what, a.C);
    if (a.stride < (long long)a.C * a.N) return mllm_fail(1, "%s: state rows of %lld floats", what, a.stride);
    if (S > 65535) return mllm_fail(1, "%s: more than 65535 requests in a step", what);
    return 0;
}

// lanes per channel, so that L * 4 (or 32 * 8) entries cover the state
int lanes_for(int N) {
    int L = 1;
    while (L < 32 && L * 4 < N) L *= 2;
    return L;
}

#define MLLM_BY_LANES(GO)                                                                                                \
    do {                                                                                                                 \
        switch (lanes_for(a.N)) {                                                                                        \
            case 1: GO(1, 4); break;                                                                                     \
            case 2: GO(2, 4); break;                                                                                     \
            case 4: GO(4, 4); break;                                                                                     \
            case 8: GO(8, 4); break;                                                                                     \
            case 16: GO(16, 4); break;                                                                                   \
            default: if (a.N <= 128) GO(32, 4); else GO(32, 8);                                                          \
        }                                                                                                                \
    } while (0)

template <typename T>
int scan_launch(const void* x, long long ldx, const float* dt, long long lddt, const void* bc, long long ldbc, int b_off, int c_off,
                const void* z, long long ldz, void* out, long long ldo, int S, const SelArgs& a, cudaStream_t stream) {
#define MLLM_GO(L, R)                                                                                                    \
    MLLM_CUDA(mllm_launch(selective_scan_kernel<T, L, R>, dim3((a.C + THREADS / L - 1) / (THREADS / L), S), dim3(2 * THREADS), 0, \
                          stream, true, (const T*)x, ldx, dt, lddt, (const T*)bc, ldbc, b_off, c_off, (const T*)z, ldz,  \
                          (T*)out, ldo, a))
    MLLM_BY_LANES(MLLM_GO);
#undef MLLM_GO
    return 0;
}

template <typename T>
int step_launch(const void* x, long long ldx, const void* low, long long ldlow, int rank, int b_off, int c_off, const void* W,
                const void* z, long long ldz, void* out, long long ldo, int S, const SelArgs& a, cudaStream_t stream) {
    const size_t smem = (size_t)((rank + 7) / 8 * 8) * 4;
#define MLLM_GO(L, R)                                                                                                    \
    MLLM_CUDA(mllm_launch(selective_step_kernel<T, L, R>, dim3((a.C + THREADS / L - 1) / (THREADS / L), S), dim3(THREADS), smem, \
                          stream, true, (const T*)x, ldx, (const T*)low, ldlow, rank, b_off, c_off, (const T*)W, (const T*)z, \
                          ldz, (T*)out, ldo, a))
    MLLM_BY_LANES(MLLM_GO);
#undef MLLM_GO
    return 0;
}

}  // namespace

MLLM_EXPORT int mllm_selective_max_state() { return 256; }
MLLM_EXPORT int mllm_selective_max_rank() { return 10240; }

MLLM_EXPORT int mllm_selective_scan(const void* x, long long ldx, const float* dt, long long lddt, const void* bc, long long ldbc,
                                    int b_off, int c_off, const void* z, long long ldz, const float* A, const float* skip,
                                    const float* bias, float* state, long long stride, const int* cu_q, const int* slots, void* out,
                                    long long ldo, int S, int C, int N, float out_scale, int write_state, int dtype,
                                    cudaStream_t stream) {
    if (S <= 0) return 0;
    SelArgs a{A, skip, bias, state, stride, cu_q, slots, C, N, write_state, out_scale};
    if (int rc = check("selective_scan", a, S)) return rc;
    for (long long ld : {ldx, lddt, ldbc, ldz, ldo})
        if (ld <= 0 || ld >= (1ll << 30)) return mllm_fail(1, "selective_scan: rows of %lld entries", ld);
    if (dtype == MLLM_F32) return scan_launch<float>(x, ldx, dt, lddt, bc, ldbc, b_off, c_off, z, ldz, out, ldo, S, a, stream);
    if (dtype == MLLM_BF16) return scan_launch<__nv_bfloat16>(x, ldx, dt, lddt, bc, ldbc, b_off, c_off, z, ldz, out, ldo, S, a, stream);
    return mllm_fail(1, "selective_scan: unknown dtype code %d", dtype);
}

MLLM_EXPORT int mllm_selective_step(const void* x, long long ldx, const void* low, long long ldlow, int rank, int b_off, int c_off,
                                    const void* W, const void* z, long long ldz, const float* A, const float* skip,
                                    const float* bias, float* state, long long stride, const int* cu_q, const int* slots, void* out,
                                    long long ldo, int S, int C, int N, float out_scale, int write_state, int dtype,
                                    cudaStream_t stream) {
    if (S <= 0) return 0;
    SelArgs a{A, skip, bias, state, stride, cu_q, slots, C, N, write_state, out_scale};
    if (int rc = check("selective_step", a, S)) return rc;
    if (rank <= 0 || rank > mllm_selective_max_rank()) return mllm_fail(1, "selective_step: step sizes of rank %d", rank);
    if ((uintptr_t)W % 16) return mllm_fail(1, "selective_step: the projection's rows must start on 16 bytes");
    if (dtype == MLLM_F32) return step_launch<float>(x, ldx, low, ldlow, rank, b_off, c_off, W, z, ldz, out, ldo, S, a, stream);
    if (dtype == MLLM_BF16) return step_launch<__nv_bfloat16>(x, ldx, low, ldlow, rank, b_off, c_off, W, z, ldz, out, ldo, S, a, stream);
    return mllm_fail(1, "selective_step: unknown dtype code %d", dtype);
}
