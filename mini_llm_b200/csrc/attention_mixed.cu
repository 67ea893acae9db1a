// Causal softmax attention over the paged cache in which the scores of a query's heads are mixed before the softmax:
//   r_g(i, j) = (q_(i,g) . k_(j, floor(g / (H / G)))) * scale        the H raw scores of query i and key j
//   s_h(i, j) = sum_g M[h, g] r_g(i, j)                              M a learned [H, H] matrix
//   p = softmax over the visible j of s_h, with exp(sink_h) added to the denominator when sinks are given
//   out_(i,h) = sum_j p_j v_(j, floor(h / (H / G)))
// Keys are visible for j <= i and, with a window w, i - j < w.  Keys and values may have different row sizes (key rows of the
// pages are padded with zeros to multiples of 8).  Every head needs every other head's raw score of the same (query, key), so
// a CTA takes all heads of a few queries.  Scores, mixing, softmax and the weighted sum are 32-bit.
//
// Two kernels.
//   rows   CUDA cores, any sizes, both cache dtypes: NQ queries of one request (1 or 4) against chunks of 64 keys that start
//          at multiples of 64 from position 0.  Raw scores: a warp takes one key/value head and 4 KG keys, 8 lanes per key
//          load its row straight into registers and take the products with all queries and heads that read it.  Mixing and
//          softmax: a warp per (query, head), two keys per lane.  Weighted sum: a warp per (key/value head, up to 4 of its
//          heads, 64 value columns, part of the keys), every value row is loaded once for all of them.
//          Single tokens (decode): grid (chunks, tokens), a chunk per CTA, partial (o, m, l) merged in chunk order by
//          `merge`; chunks before the window are not in the grid.  Prompt portions: a CTA walks its chunks.
//   mma    bfloat16 prompt portions on tensor cores (mma.sync m16n8k16): 16 queries, all heads, key tiles of 32 that start at
//          multiples of 32 from position 0.  A warp owns one head (two beyond 16 heads): its raw scores go to shared memory
//          in 32-bit, are mixed there (a thread holds a pair of keys of one query and makes the scores of 8 or 16 heads from
//          the H raw ones), come back into the warp's fragments for the online softmax, and the weights enter the second
//          product as p = hi + lo, two bfloat16 terms, so that they keep about 16 bits.
#include "common.cuh"

namespace {

constexpr int KT = 64;                  // keys per chunk of the rows kernel
constexpr int MAX_D = 256;              // largest dk and dv
constexpr int MAX_H = 64;               // most heads
constexpr int MAX_SMEM = 227 * 1024;
constexpr float LOG2E = 1.4426950408889634f;

struct MixArgs {
    const int* bt;              // block tables [requests][bt_stride]
    const int* token_seq;
    const int* positions;
    const float* mix;           // [H][H]
    const float* sink;          // [H] or null
    long long q_stride, out_stride;
    int bt_stride, H, G, dkq, dk, dv, ps, window;
    float scale;
};

__device__ __forceinline__ int first_visible(int window, int p) { return window > 0 && p - window + 1 > 0 ? p - window + 1 : 0; }

template <typename T>
__device__ __forceinline__ void unpack(const uint4& u, float* f) {      // 16 bytes: 8 bfloat16 or 4 float
    if constexpr (sizeof(T) == 4) {
        f[0] = __uint_as_float(u.x); f[1] = __uint_as_float(u.y); f[2] = __uint_as_float(u.z); f[3] = __uint_as_float(u.w);
    } else {
        f[0] = __uint_as_float(u.x << 16); f[1] = __uint_as_float(u.x & 0xffff0000u);
        f[2] = __uint_as_float(u.y << 16); f[3] = __uint_as_float(u.y & 0xffff0000u);
        f[4] = __uint_as_float(u.z << 16); f[5] = __uint_as_float(u.z & 0xffff0000u);
        f[6] = __uint_as_float(u.w << 16); f[7] = __uint_as_float(u.w & 0xffff0000u);
    }
}

// shared memory of the rows kernel, in floats: queries, mixing matrix, raw scores, weights, output sums per key part,
// (m, l, alpha) per query and head, the chunk's row numbers
__host__ __device__ __forceinline__ size_t rows_floats(int NQ, int H, int dk, int dv, int parts) {
    return (size_t)NQ * H * dk + (size_t)H * H + 2 * (size_t)NQ * H * KT + (size_t)parts * NQ * H * dv + 3 * (size_t)NQ * H + KT + 8;
}

// SPLIT: one chunk per CTA (blockIdx.x-th from the first visible one), token blockIdx.y, results to part_o / part_ml.
// Otherwise blockIdx.y is a tile (request, first flat token, rows) and the CTA takes its queries NQ * blockIdx.x ...
// U: 16-byte pieces of a key row per lane (8 lanes share a row).
template <typename T, int NQ, int U, bool SPLIT>
__global__ void __launch_bounds__(256)
attention_mixed_rows_kernel(const T* q, const T* k_pages, const T* v_pages, const int* __restrict__ tiles, T* __restrict__ out,
                            float* __restrict__ part_o, float* __restrict__ part_ml, int parts, MixArgs a) {
    constexpr int E = 16 / sizeof(T);           // elements per piece
    constexpr int KG = U <= 2 ? 4 : (U == 4 ? 2 : 1);   // groups of 4 keys a warp has in flight
    constexpr int KB = 4 * KG;                  // keys per item of the first phase
    extern __shared__ __align__(16) float sm[];
    const int H = a.H, G = a.G, R = H / G, dk = a.dk, dv = a.dv;
    float* qs = sm;                             // [NQ][H][dk], times scale
    float* Ss = qs + NQ * H * dk;               // [NQ][H][KT]
    float* Ps = Ss + NQ * H * KT;               // [NQ][H][KT]
    float* os = Ps + NQ * H * KT;               // [parts][NQ][H][dv]
    float* ml = os + parts * NQ * H * dv;       // [3][NQ][H]: m, l, alpha
    int* rowno = reinterpret_cast<int*>(ml + 3 * NQ * H);     // [KT] row of the chunk's keys in the pages (head 0), or -1
    float* Ms = reinterpret_cast<float*>(rowno + KT);         // [H][H]
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < H * H; i += 256) Ms[i] = a.mix[i];   // a weight: may be read before the kernel before this one ends
    pdl_wait();
    pdl_launch();
    int seq, tok0, nq;
    if (SPLIT) {
        tok0 = blockIdx.y;
        nq = 1;
        seq = a.token_seq[tok0];
    } else {
        const int tile = blockIdx.y;
        seq = tiles[tile * 3];
        tok0 = tiles[tile * 3 + 1] + blockIdx.x * NQ;
        nq = min(NQ, tiles[tile * 3 + 2] - (int)blockIdx.x * NQ);
        if (nq <= 0) return;
    }
    const int pos0 = a.positions[tok0], pos_max = pos0 + nq - 1;
    const int first = first_visible(a.window, pos0);
    int c_lo = first / KT, c_hi = pos_max / KT;
    if (SPLIT) {
        c_lo += blockIdx.x;
        if (c_lo > c_hi) return;                // the merge counts this token's chunks itself
        c_hi = c_lo;
    }
    const int* bt = a.bt + (size_t)seq * a.bt_stride;
    for (int i = tid; i < NQ * H * dk; i += 256) {
        const int d = i % dk, h = (i / dk) % H, n = i / (dk * H);
        qs[i] = (n < nq && d < a.dkq) ? to_f32(q[(size_t)(tok0 + n) * a.q_stride + (size_t)h * a.dkq + d]) * a.scale : 0.f;
    }
    if (!SPLIT)
        for (int i = tid; i < parts * NQ * H * dv; i += 256) os[i] = 0.f;
    for (int i = tid; i < NQ * H; i += 256) {
        const bool s = !SPLIT && a.sink;
        ml[i] = s ? a.sink[i % H] : -INFINITY;
        ml[NQ * H + i] = s ? 1.f : 0.f;
    }
    const int pieces = dk / E, sub = lane >> 3, l8 = lane & 7;
    const int cblocks = (dv + 63) / 64, hchunks = (R + 3) / 4;
    const bool v2 = dv % 2 == 0;

    for (int c = c_lo; c <= c_hi; ++c) {
        const int k0 = c * KT;
        if (tid < KT) {
            const int kp = k0 + tid;
            rowno[tid] = (kp >= first && kp <= pos_max) ? bt[kp / a.ps] * G * a.ps + kp % a.ps : -1;
        }
        __syncthreads();
        // raw scores
        for (int item = warp; item < G * (KT / KB); item += 8) {
            const int g = item % G, kb = (item / G) * KB;
            uint4 kr[KG][U];
#pragma unroll
            for (int x = 0; x < KG; ++x) {
                const int rn = rowno[kb + x * 4 + sub];
#pragma unroll
                for (int u = 0; u < U; ++u) {
                    const int pc = l8 + 8 * u;
                    kr[x][u] = make_uint4(0u, 0u, 0u, 0u);
                    if (rn >= 0 && pc < pieces)
                        kr[x][u] = *reinterpret_cast<const uint4*>(k_pages + ((size_t)rn + (size_t)g * a.ps) * dk + pc * E);
                }
            }
            for (int n = 0; n < nq; ++n) {
                for (int r = 0; r < R; ++r) {
                    const float* qr = qs + ((size_t)n * H + g * R + r) * dk;
                    float acc[KG];
#pragma unroll
                    for (int x = 0; x < KG; ++x) acc[x] = 0.f;
#pragma unroll
                    for (int u = 0; u < U; ++u) {
                        const int pc = l8 + 8 * u;
                        if (pc < pieces) {
                            float qv[E];
#pragma unroll
                            for (int e = 0; e < E; e += 4) {
                                const float4 t = *reinterpret_cast<const float4*>(qr + pc * E + e);
                                qv[e] = t.x; qv[e + 1] = t.y; qv[e + 2] = t.z; qv[e + 3] = t.w;
                            }
#pragma unroll
                            for (int x = 0; x < KG; ++x) {
                                float kv[E];
                                unpack<T>(kr[x][u], kv);
#pragma unroll
                                for (int e = 0; e < E; ++e) acc[x] = fmaf(qv[e], kv[e], acc[x]);
                            }
                        }
                    }
#pragma unroll
                    for (int x = 0; x < KG; ++x) {
                        acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], 1);
                        acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], 2);
                        acc[x] += __shfl_xor_sync(0xffffffffu, acc[x], 4);
                    }
                    float* srow = Ss + ((size_t)n * H + g * R + r) * KT + kb;
#pragma unroll
                    for (int x = 0; x < KG; ++x)
                        if (l8 == x) srow[x * 4 + sub] = acc[x];
                }
            }
        }
        __syncthreads();
        // mixing, mask, online softmax
        for (int i = warp; i < NQ * H; i += 8) {
            const int n = i / H, h = i % H;
            if (n >= nq) continue;
            const int p = pos0 + n, fv = first_visible(a.window, p);
            const float* base = Ss + (size_t)n * H * KT;
            float s0 = 0.f, s1 = 0.f;
            for (int g = 0; g < H; ++g) {
                const float m = Ms[h * H + g];
                s0 = fmaf(m, base[g * KT + lane], s0);
                s1 = fmaf(m, base[g * KT + lane + 32], s1);
            }
            const int ka = k0 + lane, kb = ka + 32;
            if (ka < fv || ka > p) s0 = -INFINITY;
            if (kb < fv || kb > p) s1 = -INFINITY;
            const float m_old = ml[i];
            const float m_new = fmaxf(m_old, warp_max(fmaxf(s0, s1)));
            const float mu = m_new == -INFINITY ? 0.f : m_new;      // no key of the chunk is seen by this query
            const float p0 = expf(s0 - mu), p1 = expf(s1 - mu), al = expf(m_old - mu);
            const float ls = warp_sum(p0 + p1);
            Ps[(size_t)i * KT + lane] = p0;
            Ps[(size_t)i * KT + lane + 32] = p1;
            __syncwarp();
            if (lane == 0) {
                ml[i] = m_new;
                ml[NQ * H + i] = ml[NQ * H + i] * al + ls;
                ml[2 * NQ * H + i] = al;
            }
        }
        __syncthreads();
        // weighted sum: item = (part of the keys, key/value head, up to 4 of its heads, 64 columns)
        const int items = parts * G * hchunks * cblocks, span = KT / parts;
        for (int item = warp; item < items; item += 8) {
            int x = item;
            const int cb = x % cblocks; x /= cblocks;
            const int hc = x % hchunks; x /= hchunks;
            const int g = x % G, part = x / G;
            const int d = cb * 64 + 2 * lane;
            const int nh = min(4, R - hc * 4), h0 = g * R + hc * 4;
            float acc[NQ][4][2];
#pragma unroll
            for (int n = 0; n < NQ; ++n)
#pragma unroll
                for (int r = 0; r < 4; ++r) acc[n][r][0] = acc[n][r][1] = 0.f;
            for (int j0 = part * span; j0 < part * span + span; j0 += 4) {
                float va[4], vb[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int rn = rowno[j0 + j];
                    va[j] = vb[j] = 0.f;
                    if (rn >= 0 && d < dv) {
                        const T* vr = v_pages + ((size_t)rn + (size_t)g * a.ps) * dv + d;
                        if (v2) {
                            if constexpr (sizeof(T) == 4) {
                                const float2 t = *reinterpret_cast<const float2*>(vr);
                                va[j] = t.x; vb[j] = t.y;
                            } else {
                                const uint32_t t = *reinterpret_cast<const uint32_t*>(vr);
                                va[j] = __uint_as_float(t << 16); vb[j] = __uint_as_float(t & 0xffff0000u);
                            }
                        } else {
                            va[j] = to_f32(vr[0]);
                            if (d + 1 < dv) vb[j] = to_f32(vr[1]);
                        }
                    }
                }
#pragma unroll
                for (int n = 0; n < NQ; ++n) {
                    if (n < nq) {
#pragma unroll
                        for (int r = 0; r < 4; ++r) {
                            if (r < nh) {
                                const float4 pj = *reinterpret_cast<const float4*>(Ps + ((size_t)n * H + h0 + r) * KT + j0);
                                acc[n][r][0] = fmaf(pj.x, va[0], acc[n][r][0]); acc[n][r][1] = fmaf(pj.x, vb[0], acc[n][r][1]);
                                acc[n][r][0] = fmaf(pj.y, va[1], acc[n][r][0]); acc[n][r][1] = fmaf(pj.y, vb[1], acc[n][r][1]);
                                acc[n][r][0] = fmaf(pj.z, va[2], acc[n][r][0]); acc[n][r][1] = fmaf(pj.z, vb[2], acc[n][r][1]);
                                acc[n][r][0] = fmaf(pj.w, va[3], acc[n][r][0]); acc[n][r][1] = fmaf(pj.w, vb[3], acc[n][r][1]);
                            }
                        }
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < NQ; ++n) {
                if (n < nq) {
#pragma unroll
                    for (int r = 0; r < 4; ++r) {
                        if (r < nh) {
                            float* o = os + (((size_t)part * NQ + n) * H + h0 + r) * dv + d;
                            const float al = SPLIT ? 0.f : ml[2 * NQ * H + n * H + h0 + r];
                            if (d < dv) o[0] = SPLIT ? acc[n][r][0] : fmaf(o[0], al, acc[n][r][0]);
                            if (d + 1 < dv) o[1] = SPLIT ? acc[n][r][1] : fmaf(o[1], al, acc[n][r][1]);
                        }
                    }
                }
            }
        }
        __syncthreads();
    }
    // the key parts meet in order
    for (int i = tid; i < nq * H * dv; i += 256) {
        const int d = i % dv, nh = i / dv, n = nh / H, h = nh % H;
        float o = 0.f;
        for (int part = 0; part < parts; ++part) o += os[(((size_t)part * NQ + n) * H + h) * dv + d];
        if (SPLIT) part_o[(((size_t)tok0 * H + h) * gridDim.x + blockIdx.x) * dv + d] = o;
        else out[(size_t)(tok0 + n) * a.out_stride + (size_t)h * dv + d] = from_f32<T>(o / ml[NQ * H + nh]);
    }
    if (SPLIT && tid < H) {
        float* o = part_ml + (((size_t)tok0 * H + tid) * gridDim.x + blockIdx.x) * 2;
        o[0] = ml[tid];
        o[1] = ml[H + tid];
    }
}

// one warp per (token, head): the chunks' partial results in chunk order, the sink's term first
template <typename T>
__global__ void __launch_bounds__(128)
attention_mixed_merge_kernel(const float* part_o, const float* part_ml, const int* __restrict__ positions, T* __restrict__ out,
                             long long out_stride, int Tn, int H, int dv, int nsplit, int window, const float* __restrict__ sink) {
    pdl_wait();
    pdl_launch();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const long long gw = (long long)blockIdx.x * 4 + warp;
    if (gw >= (long long)Tn * H) return;
    const int t = (int)(gw / H), h = (int)(gw % H);
    const int p = positions[t];
    const int used = p / KT - first_visible(window, p) / KT + 1;
    const size_t base = (size_t)gw * nsplit;
    float m = sink ? sink[h] : -INFINITY;
    for (int s = lane; s < used; s += 32) m = fmaxf(m, part_ml[(base + s) * 2]);
    m = warp_max(m);
    float l = sink ? expf(sink[h] - m) : 0.f;
    constexpr int NACC = MAX_D / 32;
    float acc[NACC];
#pragma unroll
    for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
    for (int s = 0; s < used; ++s) {
        const float f = expf(part_ml[(base + s) * 2] - m);
        l = fmaf(part_ml[(base + s) * 2 + 1], f, l);
#pragma unroll
        for (int i = 0; i < NACC; ++i) {
            const int d = lane + 32 * i;
            if (d < dv) acc[i] = fmaf(part_o[(base + s) * dv + d], f, acc[i]);
        }
    }
    T* o = out + (size_t)t * out_stride + (size_t)h * dv;
#pragma unroll
    for (int i = 0; i < NACC; ++i) {
        const int d = lane + 32 * i;
        if (d < dv) o[d] = from_f32<T>(acc[i] / l);
    }
}

// ------------------------------------------------------------------------------------------------ tensor cores
constexpr int MQ = 16, MK = 32, SLD = MK + 8;       // queries and keys per tile; row stride of the raw scores

__device__ __forceinline__ void ldsm_x4(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x2(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t* r, const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, const uint32_t* b) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool valid) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    const int n = valid ? 16 : 0;                                // 0 bytes read: the 16 bytes are zero-filled
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ uint32_t pack_bf16(float x, float y) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&v);
}
__device__ __forceinline__ float ex2(float x) {                   // 2^x in one instruction; 2^(-inf) = 0
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// bytes of shared memory: queries, `bufs` buffers of keys and values, raw scores, the mixing matrix (rows padded to HP)
__host__ __device__ __forceinline__ size_t mma_bytes(int H, int G, int dk, int dv, int bufs, int HP) {
    return (size_t)H * MQ * (dk + 8) * 2 + (size_t)bufs * G * MK * (dk + 8 + dv + 8) * 2 + (size_t)H * MQ * SLD * 4 + (size_t)H * HP * 4;
}

// NW warps, HPW heads per warp, HO mixed heads a thread makes per pass (NW * 32 / 256 groups of threads share the heads),
// NO value tiles of 8 columns the kernel is compiled for.  grid (4, tiles): a tile of up to 64 tokens is four of 16.
template <int NW, int HPW, int HO, int NO>
__global__ void __launch_bounds__(NW * 32)
attention_mixed_mma_kernel(const __nv_bfloat16* q, const __nv_bfloat16* k_pages, const __nv_bfloat16* v_pages,
                           const int* __restrict__ tiles, __nv_bfloat16* __restrict__ out, int bufs, MixArgs a) {
    using bf = __nv_bfloat16;
    constexpr int NT = NW * 32, NG = NT / 256, HP = NG * HO;    // HP: heads padded to what the groups make
    extern __shared__ __align__(16) unsigned char smraw[];
    const int H = a.H, G = a.G, R = H / G, dk = a.dk, dv = a.dv;
    const int qrow = dk + 8, vrow = dv + 8;                      // 16 bytes of padding: ldmatrix rows fall on different banks
    bf* Qs = reinterpret_cast<bf*>(smraw);                       // [H][MQ][dk + 8]
    bf* Ks = Qs + (size_t)H * MQ * qrow;                         // [bufs][G][MK][dk + 8]
    bf* Vs = Ks + (size_t)bufs * G * MK * qrow;                  // [bufs][G][MK][dv + 8]
    float* Ss = reinterpret_cast<float*>(Vs + (size_t)bufs * G * MK * vrow);     // [H][MQ][SLD]
    float* Mt = Ss + (size_t)H * MQ * SLD;                       // [H (raw)][HP (mixed)]: the mixing matrix transposed
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < H * HP; i += NT) {
        const int g = i / HP, h = i % HP;
        Mt[i] = h < H ? a.mix[h * H + g] : 0.f;
    }
    pdl_wait();
    pdl_launch();
    const int tile = blockIdx.y;
    const int rows = min(MQ, tiles[tile * 3 + 2] - (int)blockIdx.x * MQ);
    if (rows <= 0) return;
    const int seq = tiles[tile * 3], tok0 = tiles[tile * 3 + 1] + blockIdx.x * MQ;
    const int pos0 = a.positions[tok0], pos_max = pos0 + rows - 1;
    const int* bt = a.bt + (size_t)seq * a.bt_stride;
    const int first_key = first_visible(a.window, pos0);
    const int kp8 = dk / 8, vp8 = dv / 8;
    // A key's row of one key/value head (its kp8 + vp8 pieces of 16 bytes) is copied by `1 << lsh` lanes, so a thread's key,
    // head and pieces follow from shifts; lane l of a warp has looked up the page row of key l of the tile.
    const int per = kp8 + vp8, lsh = per <= 4 ? 2 : (per <= 8 ? 3 : (per <= 16 ? 4 : 5));
    const int ps_shift = (a.ps & (a.ps - 1)) == 0 ? __ffs(a.ps) - 1 : -1;       // pages of a power of two: shifts
    auto stage = [&](int j, int buf) {                           // key tile j into buffer buf
        bf* kd = Ks + (size_t)buf * G * MK * qrow;
        bf* vd = Vs + (size_t)buf * G * MK * vrow;
        int mine = -1;
        {
            const int kp = j * MK + lane;
            if (kp <= pos_max && kp >= first_key) {
                const int pg = ps_shift >= 0 ? kp >> ps_shift : kp / a.ps;
                const int off = ps_shift >= 0 ? kp & (a.ps - 1) : kp % a.ps;
                mine = bt[pg] * G * a.ps + off;
            }
        }
        for (int r = tid >> lsh; r < MK * G; r += NT >> lsh) {   // row r: key r & 31 of head r >> 5 (the same trips for a whole warp)
            const int key = r & (MK - 1), g = r >> 5;
            const int row0 = __shfl_sync(0xffffffffu, mine, key);
            const bool ok = row0 >= 0;
            const size_t rn = ok ? (size_t)row0 + (size_t)g * a.ps : 0;
            for (int piece = lane & ((1 << lsh) - 1); piece < per; piece += 1 << lsh) {
                if (piece < kp8) cp_async16(kd + (size_t)r * qrow + piece * 8, k_pages + rn * dk + piece * 8, ok);
                else cp_async16(vd + (size_t)r * vrow + (piece - kp8) * 8, v_pages + rn * dv + (piece - kp8) * 8, ok);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int i = tid; i < H * MQ * kp8; i += NT) {               // queries: rows beyond the tile are zero
        const int piece = i % kp8, r = (i / kp8) % MQ, h = i / (kp8 * MQ);
        cp_async16(Qs + ((size_t)h * MQ + r) * qrow + piece * 8,
                   r < rows ? q + (size_t)(tok0 + r) * a.q_stride + (size_t)h * dk + piece * 8 : q, r < rows);
    }
    const int j_first = first_key / MK, j_last = pos_max / MK;
    stage(j_first, 0);

    const int r0 = lane >> 2, cq = 2 * (lane & 3);               // this thread's rows r0, r0 + 8 and columns cq, cq + 1 of a fragment
    const int qp0 = pos0 + r0, qp1 = qp0 + 8;
    float o[HPW][NO][4], m0[HPW], m1[HPW], l0[HPW], l1[HPW];
#pragma unroll
    for (int x = 0; x < HPW; ++x) {
        const int h = warp * HPW + x;
#pragma unroll
        for (int i = 0; i < NO; ++i) o[x][i][0] = o[x][i][1] = o[x][i][2] = o[x][i][3] = 0.f;
        const bool s = a.sink && h < H;                          // scores in units of ln 2; one thread of a row's quad carries the sink's weight
        m0[x] = m1[x] = s ? a.sink[h] * LOG2E : -INFINITY;
        l0[x] = l1[x] = (s && (lane & 3) == 0) ? 1.f : 0.f;
    }
    const int nvt = dv / 8;
    for (int j = j_first; j <= j_last; ++j) {
        const int buf = bufs == 2 ? (j - j_first) & 1 : 0;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                         // tile j is in; the other buffer is free
        if (bufs == 2 && j < j_last) stage(j + 1, buf ^ 1);
        const bf* kt = Ks + (size_t)buf * G * MK * qrow;
        const bf* vt = Vs + (size_t)buf * G * MK * vrow;
#pragma unroll
        for (int x = 0; x < HPW; ++x) {                          // raw scores of this warp's heads
            const int h = warp * HPW + x;
            if (h >= H) continue;
            const bf* kg = kt + (size_t)(h / R) * MK * qrow;
            const bf* qh = Qs + (size_t)h * MQ * qrow;
            float s[4][4];
#pragma unroll
            for (int n = 0; n < 4; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
            for (int k0 = 0; k0 < dk; k0 += 16) {
                uint32_t af[4];
                ldsm_x4(af, qh + (lane & 15) * qrow + k0 + (lane >> 4) * 8);
#pragma unroll
                for (int n = 0; n < 4; ++n) {
                    uint32_t bfr[2];
                    ldsm_x2(bfr, kg + (n * 8 + (lane & 7)) * qrow + k0 + ((lane >> 3) & 1) * 8);
                    mma_bf16(s[n], af, bfr);
                }
            }
            float* sr = Ss + ((size_t)h * MQ + r0) * SLD + cq;
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                *reinterpret_cast<float2*>(sr + n * 8) = make_float2(s[n][0] * a.scale, s[n][1] * a.scale);
                *reinterpret_cast<float2*>(sr + 8 * SLD + n * 8) = make_float2(s[n][2] * a.scale, s[n][3] * a.scale);
            }
        }
        __syncthreads();
        {                                                        // mixing, in place: thread (pair of keys, group of heads)
            const int pair = tid & 255, grp = tid >> 8;
            float* sp = Ss + (size_t)(pair >> 4) * SLD + 2 * (pair & 15);
            float2 y[HO];
#pragma unroll
            for (int i = 0; i < HO; ++i) y[i] = make_float2(0.f, 0.f);
            for (int g = 0; g < H; ++g) {
                const float2 r = *reinterpret_cast<const float2*>(sp + (size_t)g * MQ * SLD);
                const float4* mt = reinterpret_cast<const float4*>(Mt + g * HP + grp * HO);
#pragma unroll
                for (int i = 0; i < HO / 4; ++i) {
                    const float4 w = mt[i];
                    y[4 * i].x = fmaf(w.x, r.x, y[4 * i].x); y[4 * i].y = fmaf(w.x, r.y, y[4 * i].y);
                    y[4 * i + 1].x = fmaf(w.y, r.x, y[4 * i + 1].x); y[4 * i + 1].y = fmaf(w.y, r.y, y[4 * i + 1].y);
                    y[4 * i + 2].x = fmaf(w.z, r.x, y[4 * i + 2].x); y[4 * i + 2].y = fmaf(w.z, r.y, y[4 * i + 2].y);
                    y[4 * i + 3].x = fmaf(w.w, r.x, y[4 * i + 3].x); y[4 * i + 3].y = fmaf(w.w, r.y, y[4 * i + 3].y);
                }
            }
            if (NG > 1) __syncthreads();                         // every group has read the raw scores
#pragma unroll
            for (int i = 0; i < HO; ++i) {
                const int h = grp * HO + i;
                if (h < H) *reinterpret_cast<float2*>(sp + (size_t)h * MQ * SLD) = y[i];
            }
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < HPW; ++x) {
            const int h = warp * HPW + x;
            if (h >= H) continue;
            const float* sr = Ss + ((size_t)h * MQ + r0) * SLD + cq;
            float s[4][4];
            float mx0 = -INFINITY, mx1 = -INFINITY;
            const int f0 = first_visible(a.window, qp0), f1 = first_visible(a.window, qp1);
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                const float2 u = *reinterpret_cast<const float2*>(sr + n * 8);
                const float2 w = *reinterpret_cast<const float2*>(sr + 8 * SLD + n * 8);
                const int kp = j * MK + n * 8 + cq;
                s[n][0] = (kp <= qp0 && kp >= f0) ? u.x * LOG2E : -INFINITY;
                s[n][1] = (kp + 1 <= qp0 && kp + 1 >= f0) ? u.y * LOG2E : -INFINITY;
                s[n][2] = (kp <= qp1 && kp >= f1) ? w.x * LOG2E : -INFINITY;
                s[n][3] = (kp + 1 <= qp1 && kp + 1 >= f1) ? w.y * LOG2E : -INFINITY;
                mx0 = fmaxf(mx0, fmaxf(s[n][0], s[n][1]));
                mx1 = fmaxf(mx1, fmaxf(s[n][2], s[n][3]));
            }
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            const float mn0 = fmaxf(m0[x], mx0), mn1 = fmaxf(m1[x], mx1);
            const float mu0 = mn0 == -INFINITY ? 0.f : mn0, mu1 = mn1 == -INFINITY ? 0.f : mn1;
            const float al0 = ex2(m0[x] - mu0), al1 = ex2(m1[x] - mu1);
            m0[x] = mn0; m1[x] = mn1;
            float rs0 = 0.f, rs1 = 0.f;
            uint32_t phi[2][4], plo[2][4];                       // A fragments of p for the two 16-key steps
#pragma unroll
            for (int n = 0; n < 4; ++n) {
                const float p0 = ex2(s[n][0] - mu0), p1 = ex2(s[n][1] - mu0), p2 = ex2(s[n][2] - mu1), p3 = ex2(s[n][3] - mu1);
                rs0 += p0 + p1;
                rs1 += p2 + p3;
                const __nv_bfloat162 h01 = __floats2bfloat162_rn(p0, p1), h23 = __floats2bfloat162_rn(p2, p3);
                const int kk = n >> 1, half = (n & 1) * 2;
                phi[kk][half] = *reinterpret_cast<const uint32_t*>(&h01);
                phi[kk][half + 1] = *reinterpret_cast<const uint32_t*>(&h23);
                plo[kk][half] = pack_bf16(p0 - __low2float(h01), p1 - __high2float(h01));
                plo[kk][half + 1] = pack_bf16(p2 - __low2float(h23), p3 - __high2float(h23));
            }
            l0[x] = l0[x] * al0 + rs0;                           // per-thread part of the row sums; the quad meets at the end
            l1[x] = l1[x] * al1 + rs1;
#pragma unroll
            for (int i = 0; i < NO; ++i) {
                if (i < nvt) { o[x][i][0] *= al0; o[x][i][1] *= al0; o[x][i][2] *= al1; o[x][i][3] *= al1; }
            }
            const bf* vg = vt + (size_t)(h / R) * MK * vrow;
#pragma unroll
            for (int kk = 0; kk < 2; ++kk) {
#pragma unroll
                for (int i = 0; i < NO; ++i) {
                    if (i < nvt) {
                        uint32_t bfr[2];
                        ldsm_x2_trans(bfr, vg + (kk * 16 + (lane & 15)) * vrow + i * 8);
                        mma_bf16(o[x][i], phi[kk], bfr);
                        mma_bf16(o[x][i], plo[kk], bfr);
                    }
                }
            }
        }
        if (bufs == 1 && j < j_last) {
            __syncthreads();                                     // the tile has been used
            stage(j + 1, 0);
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int x = 0; x < HPW; ++x) {
        const int h = warp * HPW + x;
        if (h >= H) continue;
        float s0 = l0[x], s1 = l1[x];
        s0 += __shfl_xor_sync(0xffffffffu, s0, 1);
        s0 += __shfl_xor_sync(0xffffffffu, s0, 2);
        s1 += __shfl_xor_sync(0xffffffffu, s1, 1);
        s1 += __shfl_xor_sync(0xffffffffu, s1, 2);
        const float inv0 = 1.0f / s0, inv1 = 1.0f / s1;
#pragma unroll
        for (int i = 0; i < NO; ++i) {
            if (i < nvt) {
                const int col = i * 8 + cq;
                if (r0 < rows)
                    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(tok0 + r0) * a.out_stride + (size_t)h * dv + col) =
                        __floats2bfloat162_rn(o[x][i][0] * inv0, o[x][i][1] * inv0);
                if (r0 + 8 < rows)
                    *reinterpret_cast<__nv_bfloat162*>(out + (size_t)(tok0 + r0 + 8) * a.out_stride + (size_t)h * dv + col) =
                        __floats2bfloat162_rn(o[x][i][2] * inv1, o[x][i][3] * inv1);
            }
        }
    }
}

int mma_padded_heads(int H) { return H <= 8 ? 8 : (H <= 16 ? 16 : 32); }

// buffers of keys and values that fit (2, 1), or 0: not a case for the tensor-core kernel
int mma_bufs(int H, int G, int dk, int dv) {
    if (H > 32 || dk % 16 != 0 || dv % 8 != 0 || dk > 128 || dv > 128) return 0;
    for (int b = 2; b >= 1; --b)
        if (mma_bytes(H, G, dk, dv, b, mma_padded_heads(H)) <= MAX_SMEM) return b;
    return 0;
}

int row_parts(int G, int R, int dv) {           // parts of a chunk's keys, so that the weighted sum has an item for every warp
    const int items = G * ((R + 3) / 4) * ((dv + 63) / 64);
    int p = 1;
    while (p * 2 * items <= 8 && p < 8) p *= 2;
    return p;
}

template <typename T, int NQ, bool SPLIT>
int launch_rows(dim3 grid, const void* q, const void* k_pages, const void* v_pages, const int* tiles, void* out, float* part_o,
                float* part_ml, const MixArgs& a, cudaStream_t stream) {
    const int parts = row_parts(a.G, a.H / a.G, a.dv);
    const size_t smem = 4 * rows_floats(NQ, a.H, a.dk, a.dv, parts);
    if (smem > MAX_SMEM) return mllm_fail(1, "attention_mixed: %d heads of %d / %d need %zu bytes of shared memory", a.H, a.dk, a.dv, smem);
    const int lanes8 = (a.dk * (int)sizeof(T) / 16 + 7) / 8;     // 16-byte pieces per lane with 8 lanes per row
#define MLLM_ROWS(UU)                                                                                                    \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            MLLM_CUDA(cudaFuncSetAttribute(attention_mixed_rows_kernel<T, NQ, UU, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        MLLM_CUDA(mllm_launch(attention_mixed_rows_kernel<T, NQ, UU, SPLIT>, grid, dim3(256), smem, stream, true, (const T*)q, \
                              (const T*)k_pages, (const T*)v_pages, tiles, (T*)out, part_o, part_ml, parts, a));          \
    } while (0)
    if (lanes8 <= 1) MLLM_ROWS(1); else if (lanes8 <= 2) MLLM_ROWS(2); else if (lanes8 <= 4) MLLM_ROWS(4); else MLLM_ROWS(8);
#undef MLLM_ROWS
    return 0;
}

template <typename T>
int run_rows(const void* q, const void* k_pages, const void* v_pages, const int* tiles, int n_tiles, void* out, float* part_o,
             float* part_ml, int nsplit, int Tn, const MixArgs& a, cudaStream_t stream) {
    if (part_o) {
        if (int rc = launch_rows<T, 1, true>(dim3(nsplit, Tn), q, k_pages, v_pages, nullptr, out, part_o, part_ml, a, stream)) return rc;
        MLLM_CUDA(mllm_launch(attention_mixed_merge_kernel<T>, dim3((unsigned)(((long long)Tn * a.H + 3) / 4)), dim3(128), 0, stream, true,
                              (const float*)part_o, (const float*)part_ml, a.positions, (T*)out, a.out_stride, Tn, a.H, a.dv, nsplit,
                              a.window, a.sink));
        return 0;
    }
    if (4 * rows_floats(4, a.H, a.dk, a.dv, row_parts(a.G, a.H / a.G, a.dv)) <= MAX_SMEM)
        return launch_rows<T, 4, false>(dim3(16, n_tiles), q, k_pages, v_pages, tiles, out, nullptr, nullptr, a, stream);
    return launch_rows<T, 1, false>(dim3(64, n_tiles), q, k_pages, v_pages, tiles, out, nullptr, nullptr, a, stream);
}

}  // namespace

MLLM_EXPORT int mllm_attention_mixed_chunk() { return KT; }

// 1 if heads of these sizes fit the CUDA-core kernel (every step can run)
MLLM_EXPORT int mllm_attention_mixed_ok(int H, int G, int dk, int dv) {
    return H >= 1 && H <= MAX_H && G >= 1 && H % G == 0 && dk >= 1 && dk <= MAX_D && dk % 8 == 0 && dv >= 1 && dv <= MAX_D &&
           4 * rows_floats(1, H, dk, dv, row_parts(G, H / G, dv)) <= MAX_SMEM;
}

// 1 if the tensor-core kernel takes these sizes (bfloat16 and aligned rows are the caller's to check)
MLLM_EXPORT int mllm_attention_mixed_mma_ok(int H, int G, int dk, int dv) { return mma_bufs(H, G, dk, dv) > 0; }

// impl: 0 rows over tiles (prompt portions), 1 rows over chunks of single tokens (needs part_o [T*H*nsplit*dv], part_ml
// [T*H*nsplit*2]; nsplit: the most chunks a token of the step sees), 2 tensor cores over tiles.
// tiles [n_tiles][3] = (request, first flat token, rows <= 64).
MLLM_EXPORT int mllm_attention_mixed(const void* q, long long q_stride, const void* k_pages, const void* v_pages, const int* bt,
                                     int bt_stride, const int* token_seq, const int* positions, const int* tiles, int n_tiles,
                                     void* out, long long out_stride, float* part_o, float* part_ml, int nsplit, int T, int H,
                                     int G, int dkq, int dk, int dv, int ps, float scale, const float* mix, int window,
                                     const float* sink, int dtype, int impl, cudaStream_t stream) {
    if (T <= 0) return 0;
    if (dtype != MLLM_F32 && dtype != MLLM_BF16) return mllm_fail(1, "attention_mixed: unknown dtype code %d", dtype);
    if (!mllm_attention_mixed_ok(H, G, dk, dv)) return mllm_fail(1, "attention_mixed: %d heads over %d, sizes %d / %d", H, G, dk, dv);
    if (dkq <= 0 || dkq > dk || ps <= 0 || window < 0 || !mix) return mllm_fail(1, "attention_mixed: queries of %d, pages of %d, window %d", dkq, ps, window);
    const int es = dtype == MLLM_F32 ? 4 : 2;
    if ((uintptr_t)k_pages % 16 != 0 || (uintptr_t)v_pages % (2 * es) != 0) return mllm_fail(1, "attention_mixed: unaligned pages");
    MixArgs a{bt, token_seq, positions, mix, sink, q_stride, out_stride, bt_stride, H, G, dkq, dk, dv, ps, window, scale};
    if (impl == 1) {
        if (!part_o || !part_ml || nsplit <= 0) return mllm_fail(1, "attention_mixed: single tokens need scratch for their partial results");
        if (T > 65535) return mllm_fail(1, "attention_mixed: more than 65535 single tokens");
    } else if (!tiles || n_tiles <= 0 || n_tiles > 65535) {
        return mllm_fail(1, "attention_mixed: prompt portions need the step's tile list");
    }
    if (impl == 0 || impl == 1) {
        if (impl == 0) part_o = part_ml = nullptr;
        return dtype == MLLM_F32
                   ? run_rows<float>(q, k_pages, v_pages, tiles, n_tiles, out, part_o, part_ml, nsplit, T, a, stream)
                   : run_rows<__nv_bfloat16>(q, k_pages, v_pages, tiles, n_tiles, out, part_o, part_ml, nsplit, T, a, stream);
    }
    if (impl != 2) return mllm_fail(1, "attention_mixed: unknown implementation %d", impl);
    const int bufs = mma_bufs(H, G, dk, dv);
    if (dtype != MLLM_BF16 || !bufs || dkq != dk || out_stride % 2 != 0 || (uintptr_t)out % 4 != 0 || (uintptr_t)v_pages % 16 != 0 ||
        (uintptr_t)q % 16 != 0 || q_stride % 8 != 0)
        return mllm_fail(1, "attention_mixed: the tensor-core kernel takes bfloat16, up to 32 heads, key sizes that are multiples of 16 "
                            "and value sizes of 8 up to 128, and 16-byte aligned rows (got %d heads of %d / %d)", H, dk, dv);
    const size_t smem = mma_bytes(H, G, dk, dv, bufs, mma_padded_heads(H));
#define MLLM_MIX(NW, HPW, HO, NO)                                                                                        \
    do {                                                                                                                 \
        if (smem > 48 * 1024)                                                                                            \
            MLLM_CUDA(cudaFuncSetAttribute(attention_mixed_mma_kernel<NW, HPW, HO, NO>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        MLLM_CUDA(mllm_launch(attention_mixed_mma_kernel<NW, HPW, HO, NO>, dim3(4, n_tiles), dim3(NW * 32), smem, stream, true, \
                              (const __nv_bfloat16*)q, (const __nv_bfloat16*)k_pages, (const __nv_bfloat16*)v_pages, tiles, \
                              (__nv_bfloat16*)out, bufs, a));                                                            \
    } while (0)
#define MLLM_MIX_NO(NW, HPW, HO)                                                                                         \
    do {                                                                                                                 \
        if (dv <= 32) MLLM_MIX(NW, HPW, HO, 4); else if (dv <= 64) MLLM_MIX(NW, HPW, HO, 8); else MLLM_MIX(NW, HPW, HO, 16); \
    } while (0)
    if (H <= 8) MLLM_MIX_NO(8, 1, 8); else if (H <= 16) MLLM_MIX_NO(16, 1, 8); else MLLM_MIX_NO(16, 2, 16);
#undef MLLM_MIX_NO
#undef MLLM_MIX
    return 0;
}
