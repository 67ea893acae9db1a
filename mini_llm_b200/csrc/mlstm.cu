// A matrix memory per head with exponential gates kept below a running maximum (the mLSTM cell of xLSTM).  Per head, with
// q_t (times qscale), k_t rows of dk entries, v_t of dv, a log input gate i_t and a log forget gate f_t,
//   i = cap * tanh(zi / cap)          f = logsigmoid(cap * tanh(zf / cap))          zi, zf: the gates' projections with bias
//   m_t = max(f_t + m_(t-1), i_t)     a_t = exp(f_t + m_(t-1) - m_t)     b_t = exp(i_t - m_t)
//   S_t = a_t S_(t-1) + b_t k_t v_t^T          n_t = a_t n_(t-1) + b_t k_t
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + deps)
//   y_t = o_t / sqrt(mean(o_t^2) + eps) * weight * sigmoid(g_t)
// S [dk, dv], n [dk] and m are zero at the start of a sequence.  The projections come in 32-bit; everything here is 32-bit.
// A request's state is one row: S of every head, then n of every head, then m of every head.
//
// Three kernels.  `step`: steps of single tokens in one launch, one CTA per (request, head).  `scan` and `finish`: steps that
// carry prompt portions.  `scan`: a CTA takes COLS columns of one (request, head)'s S; thread (column, row group) keeps WR
// rows in registers for the whole walk; tokens come 16 at a time (q, k, v by cp.async, two buffers); a warp of its own makes
// the gates a chunk ahead (a lane per token; only m runs token by token), and in the first column block further warps walk n
// and take n . q; the row groups' partial outputs meet in group order.  Every element of S and n is a recurrence of its own and m runs
// token by token, so the state after some tokens is the same bits however they were cut into steps.  `finish`: a warp per
// (token, head): the denominator, the unit norm, the weight and the gate.
#include "common.cuh"

namespace {

constexpr int CH = 16;              // tokens per chunk of the scan
constexpr int MAX_D = 256;          // largest dk and dv

struct MlstmArgs {
    const float* proj;              // [T][ld]
    long long ld;
    int q_off, k_off, v_off, g_off, i_off, f_off;
    float* state;                   // [slots][stride]: S [H][dk][dv], n [H][dk], m [H]
    long long stride;
    const int* cu_q;
    const int* slots;
    int H, dk, dv, write_state;
    float cap, qscale, deps, eps;
};

__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {      // log sigmoid(x) = min(x, 0) - log(1 + e^-|x|)
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ void cp4(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(d), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(float* dst, const float* src) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(d), "l"(src) : "memory");
}

// grid (requests, heads, column blocks).  Block: COLS * G threads (G = ceil(dk / WR) row groups) rounded up to whole warps,
// the gates' warp, then NW = ceil(dk / 32) warps that walk n (a lane per row; the first column block only).
// raw [T][H * dv]: S^T q (q not yet scaled); aux [T][H][2]: n . q and m.  vec: rows can be copied 16 bytes at a time.
template <int WR, int COLS>
__global__ void __launch_bounds__(COLS * 16 + 32 + WR * 16)
mlstm_scan_kernel(float* __restrict__ raw, float* __restrict__ aux, int vec, MlstmArgs a) {
    extern __shared__ __align__(16) float sm[];
    const int dk = a.dk, dv = a.dv, H = a.H;
    const int G = (dk + WR - 1) / WR, NW = (dk + 31) / 32, nmain = G * COLS;
    const int np = max(G * WR, NW * 32);        // rows beyond dk are zeros
    const int buf_floats = CH * (2 * np + COLS);
    float* os = sm + 2 * buf_floats;            // [G][CH][COLS]
    float2* gs = reinterpret_cast<float2*>(os + G * CH * COLS);      // [2][CH]: (a, b) of two chunks
    float* ns = reinterpret_cast<float*>(gs + 2 * CH);               // [NW][CH]: n . q of the chunk, per warp of rows
    pdl_wait();
    pdl_launch();
    const int seq = blockIdx.x, h = blockIdx.y, j0 = blockIdx.z * COLS;
    const int tid = threadIdx.x, nthreads = blockDim.x;
    const int t0 = a.cu_q[seq], n = a.cu_q[seq + 1] - t0;
    if (n <= 0) return;
    float* st = a.state + (size_t)a.slots[seq] * a.stride;
    float* Sg = st + (size_t)h * dk * dv;
    float* ng = st + (size_t)H * dk * dv + (size_t)h * dk;
    float* mg = st + (size_t)H * dk * (dv + 1) + h;
    const int gate0 = (nmain + 31) / 32 * 32, lane = tid & 31, aw = (tid - gate0) >> 5;      // aw: 0 the gates' warp, 1 .. NW those of n
    const bool main_thread = tid < nmain, gate_warp = tid >= gate0 && aw == 0, keeps_n = blockIdx.z == 0;
    const bool n_warp = tid >= gate0 && aw > 0 && keeps_n;
    const int nrow = (aw - 1) * 32 + lane;      // an n warp's row
    const int col = tid % COLS, g = tid / COLS, j = j0 + col;
    const bool live = main_thread && j < dv;
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
    float m = 0.f;                              // the gates' warp: the running maximum
    float zi = 0.f, zf = 0.f;                   // its next chunk's gate projections, a lane per token
    auto fetch_gates = [&](int c0) {
        if (lane < min(CH, n - c0)) {
            const float* row = a.proj + (size_t)(t0 + c0 + lane) * a.ld;
            zi = row[a.i_off + h];
            zf = row[a.f_off + h];
        }
    };
    auto make_gates = [&](int c0, int buf) {    // a and b of the chunk's tokens
        const int nc = min(CH, n - c0);
        const float li = log_input_gate(zi, a.cap), lf = log_forget_gate(zf, a.cap);
        float before = 0.f, after = 0.f;
#pragma unroll
        for (int c = 0; c < CH; ++c) {
            const float fc = __shfl_sync(0xffffffffu, lf, c), ic = __shfl_sync(0xffffffffu, li, c);
            if (c < nc) {
                const float fm = fc + m;
                m = fmaxf(fm, ic);
                if (lane == c) { before = fm; after = m; }
            }
        }
        if (lane < nc) {
            gs[buf * CH + lane] = make_float2(expf(before - after), expf(li - after));
            if (keeps_n) aux[((size_t)(t0 + c0 + lane) * H + h) * 2 + 1] = after;
        }
    };
    stage(0, 0);
    float s[WR];                                // a main thread's rows of its column; an n warp's row in s[0]
#pragma unroll
    for (int i = 0; i < WR; ++i) s[i] = 0.f;
    if (gate_warp) {
        m = *mg;
        fetch_gates(0);
        make_gates(0, 0);
        if (CH < n) fetch_gates(CH);
    } else if (n_warp) {
        if (nrow < dk) s[0] = ng[nrow];
    } else if (live) {
#pragma unroll
        for (int i = 0; i < WR; ++i)
            if (g * WR + i < dk) s[i] = Sg[(size_t)(g * WR + i) * dv + j];
    }
    for (int c0 = 0, buf = 0; c0 < n; c0 += CH, buf ^= 1) {
        const int nc = min(CH, n - c0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                        // this chunk and its gates are in; the other buffer and the sums are free
        const bool more = c0 + CH < n;
        if (more) stage(c0 + CH, buf ^ 1);
        const float* qd = sm + buf * buf_floats;
        const float* kd = qd + CH * np;
        const float* vd = kd + CH * np;
        const float2* ga = gs + buf * CH;
        if (main_thread) {
            auto walk = [&](int c) {
                const float2 ab = ga[c];
                const float at = ab.x, bv = ab.y * vd[c * COLS + col];
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
        } else if (gate_warp) {
            if (more) {
                make_gates(c0 + CH, buf ^ 1);
                if (c0 + 2 * CH < n) fetch_gates(c0 + 2 * CH);
            }
        } else if (n_warp) {
            float part[CH];
#pragma unroll
            for (int c = 0; c < CH; ++c) {
                part[c] = 0.f;
                if (c < nc) {
                    const float2 ab = ga[c];
                    s[0] = fmaf(ab.x, s[0], ab.y * kd[c * np + nrow]);
                    part[c] = s[0] * qd[c * np + nrow];
                }
            }
            // sums of 16 tokens over 32 lanes: at every step a lane keeps half of its tokens and hands the other half over
#pragma unroll
            for (int w = CH / 2; w >= 1; w /= 2) {
                const bool up = lane & w;
#pragma unroll
                for (int i = 0; i < w; ++i) {
                    const float keep = up ? part[i + w] : part[i], give = up ? part[i] : part[i + w];
                    part[i] = keep + __shfl_xor_sync(0xffffffffu, give, w);
                }
            }
            part[0] += __shfl_xor_sync(0xffffffffu, part[0], 16);
            if (lane < CH) ns[(aw - 1) * CH + lane] = part[0];       // lane l < 16 ends with token l
        }
        __syncthreads();
        for (int i = tid; i < nc * COLS; i += nthreads) {       // the row groups meet in group order
            const int c = i / COLS, d = i % COLS;
            if (j0 + d >= dv) continue;
            float acc = os[c * COLS + d];
            for (int gg = 1; gg < G; ++gg) acc += os[(gg * CH + c) * COLS + d];
            raw[(size_t)(t0 + c0 + c) * ((size_t)H * dv) + (size_t)h * dv + j0 + d] = acc;
        }
        if (n_warp && aw == 1 && lane < nc) {
            float nq = ns[lane];
            for (int w = 1; w < NW; ++w) nq += ns[w * CH + lane];
            aux[((size_t)(t0 + c0 + lane) * H + h) * 2] = nq;
        }
    }
    if (!a.write_state) return;
    if (live) {
#pragma unroll
        for (int i = 0; i < WR; ++i)
            if (g * WR + i < dk) Sg[(size_t)(g * WR + i) * dv + j] = s[i];
    }
    if (n_warp && nrow < dk) ng[nrow] = s[0];
    // m is written by mlstm_finish_kernel: every column block of this launch reads it
}

// the output of a head from its raw sums: denominator and unit norm (ss: the sum of raw^2 over the head's dv entries)
__device__ __forceinline__ float out_scale(float nq, float m, float ss, const MlstmArgs& a) {
    const float den = fmaxf(fabsf(nq * a.qscale), expf(-m)) + a.deps;
    const float c = a.qscale / den;             // o = raw * c
    return c / sqrtf(ss * c * c / (float)a.dv + a.eps);
}

// one warp per (token, head).  The warp of a request's last token also writes the head's m to the state: every column block
// of the scan reads it, so none of them may write it.
template <typename TO>
__global__ void __launch_bounds__(128)
mlstm_finish_kernel(const float* raw, const float* aux, const float* __restrict__ weight, const int* __restrict__ token_seq,
                    TO* __restrict__ y, long long y_stride, int Tn, MlstmArgs a) {
    pdl_wait();
    pdl_launch();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long gw = (long long)blockIdx.x * 4 + warp;
    if (gw >= (long long)Tn * a.H) return;
    const int t = (int)(gw / a.H), h = (int)(gw % a.H), dv = a.dv;
    const float* r = raw + (size_t)gw * dv;
    float ss = 0.f;
    for (int d = lane; d < dv; d += 32) ss = fmaf(r[d], r[d], ss);
    ss = warp_sum(ss);
    const float m = aux[gw * 2 + 1];
    const float c = out_scale(aux[gw * 2], m, ss, a);
    const float* z = a.proj + (size_t)t * a.ld + a.g_off + (size_t)h * dv;
    for (int d = lane; d < dv; d += 32)
        y[(size_t)t * y_stride + (size_t)h * dv + d] = from_f32<TO>(r[d] * c * weight[h * dv + d] / (1.0f + expf(-z[d])));
    if (a.write_state && lane == 0) {
        const int seq = token_seq[t];
        if (t + 1 == a.cu_q[seq + 1]) a.state[(size_t)a.slots[seq] * a.stride + (size_t)a.H * a.dk * (dv + 1) + h] = m;
    }
}

// Steps of single tokens: grid (requests, heads); thread (column j of evp, row group g) keeps RK rows of its column.  S comes
// into registers before the kernel waits for its predecessor (the state was written by an earlier step).
template <typename TO, int RK>
__global__ void __launch_bounds__(1024)
mlstm_step_kernel(const float* __restrict__ weight, TO* __restrict__ y, long long y_stride, int evp, MlstmArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float scratch[33];
    const int dk = a.dk, dv = a.dv, H = a.H, tid = threadIdx.x;
    const int G = blockDim.x / evp, j = tid % evp, g = tid / evp;
    float* qs = sm;                             // [dk]
    float* ks = qs + dk;                        // [dk]
    float* os = ks + dk;                        // [G][evp]
    const int seq = blockIdx.x, h = blockIdx.y;
    const int t0 = a.cu_q[seq], t1 = a.cu_q[seq + 1];
    if (t1 <= t0) return;
    float* st = a.state + (size_t)a.slots[seq] * a.stride;
    float* Sg = st + (size_t)h * dk * dv + j;
    float* ng = st + (size_t)H * dk * dv + (size_t)h * dk;
    float* mg = st + (size_t)H * dk * (dv + 1) + h;
    const bool col = j < dv;
    float s[RK];
#pragma unroll
    for (int i = 0; i < RK; ++i) {
        const int r = g * RK + i;
        s[i] = (col && r < dk) ? Sg[(size_t)r * dv] : 0.f;
    }
    float nv = tid < dk ? ng[tid] : 0.f;        // dk <= blockDim.x
    float m = *mg;
    pdl_wait();
    pdl_launch();
    for (int t = t0; t < t1; ++t) {
        const float* row = a.proj + (size_t)t * a.ld;
        const float li = log_input_gate(row[a.i_off + h], a.cap), fm = log_forget_gate(row[a.f_off + h], a.cap) + m;
        m = fmaxf(fm, li);
        const float at = expf(fm - m), bt = expf(li - m);
        __syncthreads();                        // the token before is no longer read
        float nq = 0.f;
        if (tid < dk) {
            const float q = row[a.q_off + (size_t)h * dk + tid], k = row[a.k_off + (size_t)h * dk + tid];
            qs[tid] = q;
            ks[tid] = k;
            nv = fmaf(at, nv, bt * k);
            nq = nv * q;
        }
        nq = block_sum(nq, scratch);            // its barriers also publish qs and ks
        const float bv = col ? bt * row[a.v_off + (size_t)h * dv + j] : 0.f;
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
        if (g == 0 && col) {                    // the row groups meet in group order
            o = os[j];
            for (int gg = 1; gg < G; ++gg) o += os[gg * evp + j];
        }
        const float ss = block_sum(o * o, scratch);
        if (g == 0 && col) {
            const float z = row[a.g_off + (size_t)h * dv + j];
            y[(size_t)t * y_stride + (size_t)h * dv + j] = from_f32<TO>(o * out_scale(nq, m, ss, a) * weight[h * dv + j] / (1.0f + expf(-z)));
        }
    }
    if (!a.write_state) return;
    if (col) {
#pragma unroll
        for (int i = 0; i < RK; ++i) {
            const int r = g * RK + i;
            if (r < dk) Sg[(size_t)r * dv] = s[i];
        }
    }
    if (tid < dk) ng[tid] = nv;
    if (tid == 0) *mg = m;
}

// threads and rows per thread of the single-token kernel, or 0 rows: not a case for it
void step_shape(int dk, int dv, int* evp, int* groups, int* rk) {
    *evp = (dv + 31) / 32 * 32;
    *rk = 0;
    if (dk > MAX_D || dv > MAX_D) return;
    for (int r = 4; r <= 16; r *= 4) {
        int g = (dk + r - 1) / r;
        while (g * *evp < dk) ++g;              // a thread for every entry of n
        if (g * *evp <= 1024) { *rk = r; *groups = g; return; }
    }
}

int check(const char* what, const MlstmArgs& a) {
    if (a.H <= 0 || a.H > 65535 || a.dk <= 0 || a.dk > MAX_D || a.dv <= 0 || a.dv > MAX_D)
        return mllm_fail(1, "%s: %d heads with states of %d x %d (at most %d x %d)", what, a.H, a.dk, a.dv, MAX_D, MAX_D);
    if (a.stride < (long long)a.H * (a.dk * (a.dv + 1) + 1)) return mllm_fail(1, "%s: state rows of %lld floats", what, a.stride);
    if (!(a.cap > 0.f)) return mllm_fail(1, "%s: a cap of %g on the gates", what, (double)a.cap);
    return 0;
}

}  // namespace

MLLM_EXPORT int mllm_mlstm_max_dim() { return MAX_D; }

MLLM_EXPORT int mllm_mlstm_step_ok(int dk, int dv) {
    int evp, g, rk;
    step_shape(dk, dv, &evp, &g, &rk);
    return rk > 0;
}

// proj [T][ld] 32-bit with q, k [H*dk], v, g [H*dv], i, f [H] at the given columns; state as above; raw [T][H*dv], aux
// [T][H][2] 32-bit.  want_cols: columns of S per CTA, 16 or 32, or 0 for the rule below (the same bits either way).
MLLM_EXPORT int mllm_mlstm_scan(const float* proj, long long ld, int q_off, int k_off, int v_off, int i_off, int f_off, float* state,
                                long long stride, const int* cu_q, const int* slots, float* raw, float* aux, int S, int H, int dk,
                                int dv, float cap, int write_state, int want_cols, cudaStream_t stream) {
    if (S <= 0) return 0;
    MlstmArgs a{proj, ld, q_off, k_off, v_off, 0, i_off, f_off, state, stride, cu_q, slots, H, dk, dv, write_state, cap, 1.f, 0.f, 0.f};
    if (int rc = check("mlstm_scan", a)) return rc;
    if (want_cols != 0 && want_cols != 16 && want_cols != 32) return mllm_fail(1, "mlstm_scan: %d columns per CTA (16, 32, or 0 for the rule)", want_cols);
    static int sms = 0;
    if (!sms) {
        int dev = 0;
        MLLM_CUDA(cudaGetDevice(&dev));
        MLLM_CUDA(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
    }
    // every CTA is one chain of dependent token steps: narrower CTAs shorten it as long as they all run at once
    const int cols = want_cols ? want_cols : ((dv > 16 && (long long)S * H * ((dv + 15) / 16) <= sms) ? 16 : 32);
    const int WR = dk <= 64 ? 4 : (dk <= 128 ? 8 : 16);
    const int G = (dk + WR - 1) / WR, NW = (dk + 31) / 32, np = G * WR > NW * 32 ? G * WR : NW * 32;
    const size_t smem = sizeof(float) * (2 * (size_t)CH * (2 * np + cols) + (size_t)G * CH * cols + 4 * CH + (size_t)NW * CH);
    const int vec = dk % 4 == 0 && dv % 4 == 0 && ld % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 && (uintptr_t)proj % 16 == 0;
    const dim3 grid(S, H, (dv + cols - 1) / cols), block((cols * G + 31) / 32 * 32 + 32 + 32 * NW);
#define MLLM_SCAN(WRR, CC)                                                                                               \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            MLLM_CUDA(cudaFuncSetAttribute(mlstm_scan_kernel<WRR, CC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        MLLM_CUDA(mllm_launch(mlstm_scan_kernel<WRR, CC>, grid, block, smem, stream, true, raw, aux, vec, a));           \
    } while (0)
#define MLLM_SCAN_C(WRR) do { if (cols == 16) MLLM_SCAN(WRR, 16); else MLLM_SCAN(WRR, 32); } while (0)
    if (WR == 4) MLLM_SCAN_C(4); else if (WR == 8) MLLM_SCAN_C(8); else MLLM_SCAN_C(16);
#undef MLLM_SCAN_C
#undef MLLM_SCAN
    return 0;
}

// y [T][y_stride] in `dtype` from the scan's raw and aux; weight [H*dv]; writes every request's m to its state.
MLLM_EXPORT int mllm_mlstm_finish(const float* raw, const float* aux, const float* proj, long long ld, int g_off, const float* weight,
                                  float* state, long long stride, const int* token_seq, const int* cu_q, const int* slots, void* y,
                                  long long y_stride, int T, int H, int dk, int dv, float qscale, float deps, float eps,
                                  int write_state, int dtype, cudaStream_t stream) {
    if (T <= 0) return 0;
    MlstmArgs a{proj, ld, 0, 0, 0, g_off, 0, 0, state, stride, cu_q, slots, H, dk, dv, write_state, 1.f, qscale, deps, eps};
    if (int rc = check("mlstm_finish", a)) return rc;
    const long long blocks = ((long long)T * H + 3) / 4;
    if (blocks > 2147483647LL) return mllm_fail(1, "mlstm_finish: too many (token, head) pairs");
    if (dtype == MLLM_F32)
        MLLM_CUDA(mllm_launch(mlstm_finish_kernel<float>, dim3((unsigned)blocks), dim3(128), 0, stream, true, raw, aux, weight, token_seq,
                              (float*)y, y_stride, T, a));
    else if (dtype == MLLM_BF16)
        MLLM_CUDA(mllm_launch(mlstm_finish_kernel<__nv_bfloat16>, dim3((unsigned)blocks), dim3(128), 0, stream, true, raw, aux, weight,
                              token_seq, (__nv_bfloat16*)y, y_stride, T, a));
    else
        return mllm_fail(1, "mlstm_finish: unknown dtype code %d", dtype);
    return 0;
}

// Steps of single tokens: gates, state, output, norm and gate in one launch.
MLLM_EXPORT int mllm_mlstm_step(const float* proj, long long ld, int q_off, int k_off, int v_off, int g_off, int i_off, int f_off,
                                float* state, long long stride, const int* cu_q, const int* slots, const float* weight, void* y,
                                long long y_stride, int S, int H, int dk, int dv, float cap, float qscale, float deps, float eps,
                                int write_state, int dtype, cudaStream_t stream) {
    if (S <= 0) return 0;
    MlstmArgs a{proj, ld, q_off, k_off, v_off, g_off, i_off, f_off, state, stride, cu_q, slots, H, dk, dv, write_state, cap, qscale, deps, eps};
    if (int rc = check("mlstm_step", a)) return rc;
    int evp, G = 0, rk;
    step_shape(dk, dv, &evp, &G, &rk);
    if (!rk) return mllm_fail(1, "mlstm_step: states of %d x %d", dk, dv);
    const size_t smem = sizeof(float) * (2 * (size_t)dk + (size_t)G * evp);
    const dim3 grid(S, H), block(evp * G);
#define MLLM_STEP(TT, RKK)                                                                                               \
    MLLM_CUDA(mllm_launch(mlstm_step_kernel<TT, RKK>, grid, block, smem, stream, true, weight, (TT*)y, y_stride, evp, a))
    if (dtype == MLLM_F32) {
        if (rk == 4) MLLM_STEP(float, 4); else MLLM_STEP(float, 16);
    } else if (dtype == MLLM_BF16) {
        if (rk == 4) MLLM_STEP(__nv_bfloat16, 4); else MLLM_STEP(__nv_bfloat16, 16);
    } else {
        return mllm_fail(1, "mlstm_step: unknown dtype code %d", dtype);
    }
#undef MLLM_STEP
    return 0;
}
