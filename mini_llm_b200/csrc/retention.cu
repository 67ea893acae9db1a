// Retention (RetNet): a matrix memory S [dk, dv] per head that forgets at a constant rate a_h.  With turned rows q, k of dk
// entries, v of dv and a gate row g, token after token from S = 0:
//   S <- a_h S + k v^T          o = S^T q          y = o / sqrt(mean(o^2) + eps) * silu(g)
// The projections come in 32-bit; everything here is 32-bit.  A request's state is S of every head in one row.
//
// `rotate_heads` turns the first rot_dims entries of every query and key head by position * freq[i] in place (entry i pairs
// with i + rot_dims / 2, or neighbours with `interleaved`) and multiplies the keys by a constant.  `scan` and `finish`: steps
// that carry prompt portions.  `scan`: a CTA takes COLS columns of one (request, head)'s S; thread (column, row group) keeps
// WR rows in registers for the whole walk; tokens come 16 at a time by cp.async (two buffers); the row groups' partial
// outputs meet in group order.  `step`: steps of single tokens in one launch (rotation, state, norm, gate), one CTA per
// (request, head).  Every element of S is a recurrence of its own, so the state after some tokens is the same bits however
// they were cut into steps.
#include "common.cuh"

namespace {

constexpr int CH = 16;              // tokens per chunk of the scan
constexpr int MAX_D = 256;          // largest dk and dv

struct RetArgs {
    const float* proj;              // [T][ld]
    long long ld;
    int q_off, k_off, v_off, g_off;
    const float* decay;             // [H]
    float* state;                   // [slots][stride]: S [H][dk][dv]
    long long stride;
    const int* cu_q;
    const int* slots;
    int H, dk, dv, write_state;
    float eps;
};

struct RotArgs {
    const float* freq;              // [dims / 2]
    int dims, interleaved;
    float k_scale;
};

__device__ __forceinline__ void cp4(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// entry d of a head: its partner in the rotation, the pair's number, and whether it is the pair's first
__device__ __forceinline__ void pair_of(int d, int dims, int interleaved, int* partner, int* fi, bool* first) {
    const int half = dims / 2;
    *partner = interleaved ? (d ^ 1) : (d < half ? d + half : d - half);
    *fi = interleaved ? (d >> 1) : (d < half ? d : d - half);
    *first = interleaved ? !(d & 1) : d < half;
}

// one CTA per token
__global__ void __launch_bounds__(256)
rotate_heads_kernel(float* proj, long long ld, int q_off, int k_off, int H, int dk, RotArgs r, const int* positions) {
    extern __shared__ float2 turn[];            // [dims / 2]: cos, sin
    pdl_wait();
    pdl_launch();
    float* row = proj + (size_t)blockIdx.x * ld;
    const int half = r.dims / 2, per = half + (dk - r.dims);
    const float p = (float)positions[blockIdx.x];
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
        float sn, cs;
        sincosf(p * r.freq[i], &sn, &cs);
        turn[i] = make_float2(cs, sn);
    }
    __syncthreads();
    for (int i = threadIdx.x; i < 2 * H * per; i += blockDim.x) {
        const bool key = i >= H * per;
        const int j = key ? i - H * per : i, h = j / per, e = j % per;
        float* x = row + (key ? k_off : q_off) + h * dk;
        const float sc = key ? r.k_scale : 1.0f;
        if (e >= half) {
            if (key) x[r.dims + e - half] *= sc;
            continue;
        }
        const int a = r.interleaved ? 2 * e : e, b = r.interleaved ? 2 * e + 1 : e + half;
        const float u = x[a], v = x[b];
        const float2 t = turn[e];
        x[a] = (u * t.x - v * t.y) * sc;
        x[b] = (v * t.x + u * t.y) * sc;
    }
}

// grid (requests, heads, column blocks); block COLS * G threads, G = ceil(dk / WR) row groups.  raw [T][H * dv].
template <int WR, int COLS>
__global__ void __launch_bounds__(COLS * 16)
retention_scan_kernel(float* __restrict__ raw, int vec, RetArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int dk = a.dk, dv = a.dv, H = a.H;
    const int G = (dk + WR - 1) / WR, np = G * WR;      // rows beyond dk are zeros
    const int buf_floats = CH * (2 * np + COLS);
    float* os = sm + 2 * buf_floats;            // [G][CH][COLS]
    const int seq = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, nthreads = blockDim.x;
    const float at = a.decay[h];
    pdl_wait();
    pdl_launch();
    const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
    if (n <= 0) return;
    float* Sg = a.state + (size_t)a.slots[seq] * a.stride + (size_t)h * dk * dv;
    const int col = tid % COLS, g = tid / COLS, j = j0 + col;
    const bool live = j < dv;
    // padded rows of q and k in both buffers are zero and stay zero
    for (int i = tid; i < 2 * CH * (np - dk); i += nthreads) {
        const int r = i % (np - dk), c = (i / (np - dk)) % CH, b = i / ((np - dk) * CH);
        float* base = sm + b * buf_floats + c * np + dk + r;
        base[0] = 0.f;
        base[CH * np] = 0.f;
    }
    auto stage = [&](int c0, int buf) {
        const int nc = min(CH, n - c0);
        float* qd = sm + buf * buf_floats;
        float* kd = qd + CH * np;
        float* vd = kd + CH * np;
        const float* src = a.proj + (size_t)(t0 + c0) * a.ld;
        if (vec) {
            const int p = dk / 4, pv = COLS / 4;
            for (int i = tid; i < nc * p; i += nthreads) {
                const int c = i / p, e = (i - c * p) * 4;
                const float* row = src + (size_t)c * a.ld + (size_t)h * dk + e;
                cp16(qd + c * np + e, row + a.q_off);
                cp16(kd + c * np + e, row + a.k_off);
            }
            for (int i = tid; i < nc * pv; i += nthreads) {
                const int c = i / pv, e = (i % pv) * 4;
                if (j0 + e < dv) cp16(vd + c * COLS + e, src + (size_t)c * a.ld + a.v_off + (size_t)h * dv + j0 + e);
            }
        } else {
            for (int i = tid; i < nc * dk; i += nthreads) {
                const int c = i / dk, e = i - c * dk;
                const float* row = src + (size_t)c * a.ld + (size_t)h * dk + e;
                cp4(qd + c * np + e, row + a.q_off);
                cp4(kd + c * np + e, row + a.k_off);
            }
            for (int i = tid; i < nc * COLS; i += nthreads) {
                const int c = i / COLS, e = i % COLS;
                if (j0 + e < dv) cp4(vd + i, src + (size_t)c * a.ld + a.v_off + (size_t)h * dv + j0 + e);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0, 0);
    float s[WR];
#pragma unroll
    for (int i = 0; i < WR; ++i) s[i] = live && g * WR + i < dk ? Sg[(size_t)(g * WR + i) * dv + j] : 0.f;
    for (int c0 = 0, buf = 0; c0 < n; c0 += CH, buf ^= 1) {
        const int nc = min(CH, n - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                        // this chunk is in; the other buffer and the sums are free
        if (c0 + CH < n) stage(c0 + CH, buf ^ 1);
        const float* qd = sm + buf * buf_floats;
        const float* kd = qd + CH * np;
        const float* vd = kd + CH * np;
        auto walk = [&](int c) {
            const float bv = vd[c * COLS + col];
            const float4* q4 = reinterpret_cast<const float4*>(qd + c * np + g * WR);
            const float4* k4 = reinterpret_cast<const float4*>(kd + c * np + g * WR);
            float acc0 = 0.f, acc1 = 0.f;
#pragma unroll
            for (int i = 0; i < WR / 4; ++i) {
                const float4 q = q4[i], k = k4[i];
                s[4 * i] = fmaf(at, s[4 * i], k.x * bv);
                acc0 = fmaf(s[4 * i], q.x, acc0);
                s[4 * i + 1] = fmaf(at, s[4 * i + 1], k.y * bv);
                acc1 = fmaf(s[4 * i + 1], q.y, acc1);
                s[4 * i + 2] = fmaf(at, s[4 * i + 2], k.z * bv);
                acc0 = fmaf(s[4 * i + 2], q.z, acc0);
                s[4 * i + 3] = fmaf(at, s[4 * i + 3], k.w * bv);
                acc1 = fmaf(s[4 * i + 3], q.w, acc1);
            }
            os[(g * CH + c) * COLS + col] = acc0 + acc1;
        };
        if (nc == CH) {
#pragma unroll 4
            for (int c = 0; c < CH; ++c) walk(c);
        } else {
            for (int c = 0; c < nc; ++c) walk(c);
        }
        __syncthreads();
        for (int i = tid; i < nc * COLS; i += nthreads) {       // the row groups meet in group order
            const int c = i / COLS, d = i % COLS;
            if (j0 + d >= dv) continue;
            float acc = os[c * COLS + d];
            for (int gg = 1; gg < G; ++gg) acc += os[(gg * CH + c) * COLS + d];
            raw[(size_t)(t0 + c0 + c) * ((size_t)H * dv) + (size_t)h * dv + j0 + d] = acc;
        }
    }
    if (a.write_state && live) {
#pragma unroll
        for (int i = 0; i < WR; ++i)
            if (g * WR + i < dk) Sg[(size_t)(g * WR + i) * dv + j] = s[i];
    }
}

// one warp per (token, head)
template <typename TO>
__global__ void __launch_bounds__(128)
retention_finish_kernel(const float* raw, TO* __restrict__ y, long long y_stride, int Tn, RetArgs a) {
    pdl_wait();
    pdl_launch();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long gw = (long long)blockIdx.x * 4 + warp;
    if (gw >= (long long)Tn * a.H) return;
    const int t = (int)(gw / a.H), h = (int)(gw % a.H), dv = a.dv;
    const float* r = raw + (size_t)gw * dv;
    const float* z = a.proj + (size_t)t * a.ld + a.g_off + (size_t)h * dv;
    float o[MAX_D / 32], gz[MAX_D / 32], ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
        const int d = lane + 32 * i;
        o[i] = d < dv ? r[d] : 0.f;
        gz[i] = d < dv ? z[d] : 0.f;
        ss = fmaf(o[i], o[i], ss);
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + a.eps);
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
        const int d = lane + 32 * i;
        if (d < dv) y[(size_t)t * y_stride + (size_t)h * dv + d] = from_f32<TO>(o[i] * inv * (gz[i] / (1.0f + expf(-gz[i]))));
    }
}

// Steps of single tokens: grid (requests, heads); thread (column j of evp, row group g) keeps RK rows of its column.  S comes
// into registers before the kernel waits for its predecessor (the state was written by an earlier step).
template <typename TO, int RK>
__global__ void __launch_bounds__(1024)
retention_step_kernel(TO* __restrict__ y, long long y_stride, int evp, const int* positions, RotArgs rot, RetArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[33];
    const int dk = a.dk, dv = a.dv, tid = threadIdx.x;
    const int G = blockDim.x / evp, j = tid % evp, g = tid / evp;
    float* qs = sm;                             // [dk]
    float* ks = qs + dk;                        // [dk]
    float* os = ks + dk;                        // [G][evp]
    const int seq = blockIdx.x, h = blockIdx.y;
    const int t = a.cu_q[seq];
    float* Sg = a.state + (size_t)a.slots[seq] * a.stride + (size_t)h * dk * dv + j;
    const bool col = j < dv;
    float s[RK];
#pragma unroll
    for (int i = 0; i < RK; ++i) {
        const int r = g * RK + i;
        s[i] = (col && r < dk) ? Sg[(size_t)r * dv] : 0.f;
    }
    const float at = a.decay[h], p = (float)positions[t];
    float cs = 1.f, sn = 0.f;
    int partner = 0, fi = 0;
    bool first = true;
    if (tid < dk && tid < rot.dims) {           // dk <= blockDim.x
        pair_of(tid, rot.dims, rot.interleaved, &partner, &fi, &first);
        sincosf(p * rot.freq[fi], &sn, &cs);
        if (first) sn = -sn;
    }
    pdl_wait();
    pdl_launch();
    const float* row = a.proj + (size_t)t * a.ld;
    if (tid < dk) {
        const float* q = row + a.q_off + (size_t)h * dk;
        const float* k = row + a.k_off + (size_t)h * dk;
        float qv = q[tid], kv = k[tid];
        if (tid < rot.dims) {
            qv = qv * cs + q[partner] * sn;
            kv = kv * cs + k[partner] * sn;
        }
        qs[tid] = qv;
        ks[tid] = kv * rot.k_scale;
    }
    const float bv = col ? row[a.v_off + (size_t)h * dv + j] : 0.f;
    const float z = (g == 0 && col) ? row[a.g_off + (size_t)h * dv + j] : 0.f;
    __syncthreads();
    float acc = 0.f;
#pragma unroll
    for (int i = 0; i < RK; ++i) {
        const int r = g * RK + i;
        if (r < dk) {
            s[i] = fmaf(at, s[i], ks[r] * bv);
            acc = fmaf(s[i], qs[r], acc);
        }
    }
    os[g * evp + j] = acc;
    __syncthreads();
    float o = 0.f;
    if (g == 0 && col) {                        // the row groups meet in group order
        o = os[j];
        for (int gg = 1; gg < G; ++gg) o += os[gg * evp + j];
    }
    const float inv = 1.0f / sqrtf(block_sum(o * o, scratch) / (float)dv + a.eps);
    if (g == 0 && col) y[(size_t)t * y_stride + (size_t)h * dv + j] = from_f32<TO>(o * inv * (z / (1.0f + expf(-z))));
    if (a.write_state && col) {
#pragma unroll
        for (int i = 0; i < RK; ++i) {
            const int r = g * RK + i;
            if (r < dk) Sg[(size_t)r * dv] = s[i];
        }
    }
}

// threads and rows per thread of the single-token kernel, or 0 rows: not a case for it
void step_shape(int dk, int dv, int* evp, int* groups, int* rk) {
    *evp = (dv + 31) / 32 * 32;
    *rk = 0;
    if (dk > MAX_D || dv > MAX_D) return;
    for (int r : {4, 16, 32}) {
        int g = (dk + r - 1) / r;
        while (g * *evp < dk) ++g;              // a thread for every entry of q and k
        if (g * *evp <= 1024) { *rk = r; *groups = g; return; }
    }
}

int check(const char* what, const RetArgs& a) {
    if (a.H <= 0 || a.H > 65535 || a.dk <= 0 || a.dk > MAX_D || a.dv <= 0 || a.dv > MAX_D)
        return mllm_fail(1, "%s: %d heads with states of %d x %d (at most %d x %d)", what, a.H, a.dk, a.dv, MAX_D, MAX_D);
    if (a.stride < (long long)a.H * a.dk * a.dv) return mllm_fail(1, "%s: state rows of %lld floats", what, a.stride);
    return 0;
}

int check_rot(const char* what, const RotArgs& r, int dk) {
    if (r.dims < 0 || r.dims % 2 || r.dims > dk || (r.dims > 0 && !r.freq)) return mllm_fail(1, "%s: %d rotated entries of %d", what, r.dims, dk);
    return 0;
}

}  // namespace

MLLM_EXPORT int mllm_retention_max_dim() { return MAX_D; }

MLLM_EXPORT int mllm_retention_step_ok(int dk, int dv) {
    int evp, g, rk;
    step_shape(dk, dv, &evp, &g, &rk);
    return rk > 0;
}

// In place: the query and key heads of proj [T][ld] (32-bit) turned by their token's position, the keys times k_scale.
MLLM_EXPORT int mllm_rotate_heads(float* proj, long long ld, int q_off, int k_off, int H, int dk, const float* freq, int dims,
                                  int interleaved, float k_scale, const int* positions, int T, cudaStream_t stream) {
    if (T <= 0) return 0;
    RotArgs r{freq, dims, interleaved, k_scale};
    if (H <= 0 || dk <= 0) return mllm_fail(1, "rotate_heads: %d heads of %d", H, dk);
    if (int rc = check_rot("rotate_heads", r, dk)) return rc;
    if (dims > 8192) return mllm_fail(1, "rotate_heads: %d rotated entries", dims);
    MLLM_CUDA(mllm_launch(rotate_heads_kernel, dim3(T), dim3(256), (size_t)(dims / 2) * 8, stream, true, proj, ld, q_off, k_off, H, dk,
                          r, positions));
    return 0;
}

// proj [T][ld] 32-bit with q, k [H*dk] (rotated) and v [H*dv] at the given columns; raw [T][H*dv] 32-bit.  want_cols: columns
// of S per CTA, 16 or 32, or 0 for the rule below (the same bits either way).
MLLM_EXPORT int mllm_retention_scan(const float* proj, long long ld, int q_off, int k_off, int v_off, const float* decay, float* state,
                                    long long stride, const int* cu_q, const int* slots, float* raw, int S, int H, int dk, int dv,
                                    int write_state, int want_cols, cudaStream_t stream) {
    if (S <= 0) return 0;
    RetArgs a{proj, ld, q_off, k_off, v_off, 0, decay, state, stride, cu_q, slots, H, dk, dv, write_state, 0.f};
    if (int rc = check("retention_scan", a)) return rc;
    if (want_cols != 0 && want_cols != 16 && want_cols != 32) return mllm_fail(1, "retention_scan: %d columns per CTA (16, 32, or 0 for the rule)", want_cols);
    static int sms = 0;
    if (!sms) {
        int dev = 0;
        MLLM_CUDA(cudaGetDevice(&dev));
        MLLM_CUDA(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
    }
    // every CTA is one chain of dependent token steps: narrower CTAs shorten it as long as they all run at once
    const int cols = want_cols ? want_cols : ((dv > 16 && (long long)S * H * ((dv + 15) / 16) <= sms) ? 16 : 32);
    const int WR = dk <= 64 ? 4 : (dk <= 128 ? 8 : 16);
    const int G = (dk + WR - 1) / WR, np = G * WR;
    const size_t smem = sizeof(float) * (2 * (size_t)CH * (2 * np + cols) + (size_t)G * CH * cols);
    const int vec = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 && (uintptr_t)proj % 16 == 0;
    const dim3 grid(S, H, (dv + cols - 1) / cols), block(cols * G);
#define MLLM_SCAN(WRR, CC)                                                                                               \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            MLLM_CUDA(cudaFuncSetAttribute(retention_scan_kernel<WRR, CC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        MLLM_CUDA(mllm_launch(retention_scan_kernel<WRR, CC>, grid, block, smem, stream, true, raw, vec, a));            \
    } while (0)
#define MLLM_SCAN_C(WRR) do { if (cols == 16) MLLM_SCAN(WRR, 16); else MLLM_SCAN(WRR, 32); } while (0)
    if (WR == 4) MLLM_SCAN_C(4); else if (WR == 8) MLLM_SCAN_C(8); else MLLM_SCAN_C(16);
#undef MLLM_SCAN_C
#undef MLLM_SCAN
    return 0;
}

// y [T][y_stride] in `dtype` from the scan's raw sums and the gate columns of proj.
MLLM_EXPORT int mllm_retention_finish(const float* raw, const float* proj, long long ld, int g_off, void* y, long long y_stride, int T,
                                      int H, int dv, float eps, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    RetArgs a{proj, ld, 0, 0, 0, g_off, nullptr, nullptr, 0, nullptr, nullptr, H, 0, dv, 0, eps};
    if (H <= 0 || dv <= 0 || dv > MAX_D) return mllm_fail(1, "retention_finish: %d heads of %d", H, dv);
    const long long blocks = ((long long)T * H + 3) / 4;
    if (blocks > 2147483647LL) return mllm_fail(1, "retention_finish: too many (token, head) pairs");
    if (dtype == MLLM_F32)
        MLLM_CUDA(mllm_launch(retention_finish_kernel<float>, dim3((unsigned)blocks), dim3(128), 0, stream, true, raw, (float*)y, y_stride, T, a));
    else if (dtype == MLLM_BF16)
        MLLM_CUDA(mllm_launch(retention_finish_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(128), 0, stream, true, raw,
                              (__nv_bfloat16*)y, y_stride, T, a));
    else
        return mllm_fail(1, "retention_finish: unknown dtype code %d", dtype);
    return 0;
}

// Steps of single tokens: rotation, state, output, norm and gate in one launch; proj is not yet rotated.
MLLM_EXPORT int mllm_retention_step(const float* proj, long long ld, int q_off, int k_off, int v_off, int g_off, const float* decay,
                                    const float* freq, int dims, int interleaved, float k_scale, const int* positions, float* state,
                                    long long stride, const int* cu_q, const int* slots, void* y, long long y_stride, int S, int H,
                                    int dk, int dv, float eps, int write_state, int dtype, cudaStream_t stream) {
    if (S <= 0) return 0;
    RetArgs a{proj, ld, q_off, k_off, v_off, g_off, decay, state, stride, cu_q, slots, H, dk, dv, write_state, eps};
    RotArgs r{freq, dims, interleaved, k_scale};
    if (int rc = check("retention_step", a)) return rc;
    if (int rc = check_rot("retention_step", r, dk)) return rc;
    int evp, G = 0, rk;
    step_shape(dk, dv, &evp, &G, &rk);
    if (!rk) return mllm_fail(1, "retention_step: states of %d x %d", dk, dv);
    const size_t smem = sizeof(float) * (2 * (size_t)dk + (size_t)G * evp);
    const dim3 grid(S, H), block(evp * G);
#define MLLM_STEP(TT, RKK)                                                                                               \
    MLLM_CUDA(mllm_launch(retention_step_kernel<TT, RKK>, grid, block, smem, stream, true, (TT*)y, y_stride, evp, positions, r, a))
    if (dtype == MLLM_F32) {
        if (rk == 4) MLLM_STEP(float, 4); else if (rk == 16) MLLM_STEP(float, 16); else MLLM_STEP(float, 32);
    } else if (dtype == MLLM_BF16) {
        if (rk == 4) MLLM_STEP(__nv_bfloat16, 4); else if (rk == 16) MLLM_STEP(__nv_bfloat16, 16); else MLLM_STEP(__nv_bfloat16, 32);
    } else {
        return mllm_fail(1, "retention_step: unknown dtype code %d", dtype);
    }
#undef MLLM_STEP
    return 0;
}
