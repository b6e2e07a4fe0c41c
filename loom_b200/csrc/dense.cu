// dense.cu -- 16-bit / 32-bit float matrices: storage (loom_b200_matrix_*), the small-batch GEMV and the plain token-block
// GEMM for 32-bit floats.  The bf16 token-block GEMM on the tensor cores is in gemm_bf16.cu.
#include "dense.cuh"

#include <vector>

namespace {

constexpr int kGemvThreads = 256;
constexpr int kGemvWarps = kGemvThreads / 32;
constexpr size_t kGemvSmemX = 200 * 1024;

// one thread per 16-byte chunk of the source rows
template <typename WT>
__global__ void lb_image_put_kernel(const void* __restrict__ src, int src_dtype, int rows, int cols, int row0, int slices, uint8_t* __restrict__ img) {
    constexpr int C = LbElem<WT>::kChunk;
    const int chunks = slices * 8;
    const size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (size_t)rows * chunks) return;
    const int r = (int)(idx / chunks), c = (int)(idx % chunks);
    float f[C];
#pragma unroll
    for (int i = 0; i < C; ++i) {
        const int col = c * C + i;
        float v = 0.f;
        if (col < cols)
            v = src_dtype == LOOM_B200_DTYPE_BF16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(src)[(size_t)r * cols + col])
                                                  : static_cast<const float*>(src)[(size_t)r * cols + col];
        f[i] = v;
    }
    *reinterpret_cast<uint4*>(img + lb_img_chunk(row0 + r, c, slices)) = lb_pack_chunk<WT>(f);
}

// ---- GEMV -------------------------------------------------------------------------------------------------

__device__ __forceinline__ uint4 ldg_stream(const uint8_t* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ void mma_bf16(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// Accumulator of a warp's 16 rows.  bf16: the m16n8 fragment of lane (g, t) = rows g, g+8 x tokens 2t, 2t+1.  float: rows
// g, g+8 x all eight tokens, over the K chunks of lane column t (summed over t at the end).
template <typename WT>
struct GemvAcc;
template <>
struct GemvAcc<__nv_bfloat16> {
    float d[4];
    __device__ __forceinline__ void zero() { d[0] = d[1] = d[2] = d[3] = 0.f; }
    // one 16-byte chunk of rows g and g+8 against the same chunk of token g: which two k of a chunk an MMA takes as its
    // "low" and "high" pair is the same for both operands, so the order inside the chunk cancels
    __device__ __forceinline__ void step(const uint4& w0, const uint4& w1, const uint4* xs, int Mp, int M, int g) {
        const uint4 x = g < Mp ? xs[g] : make_uint4(0, 0, 0, 0);
        mma_bf16(d, w0.x, w1.x, w0.y, w1.y, x.x, x.y);
        mma_bf16(d, w0.z, w1.z, w0.w, w1.w, x.z, x.w);
    }
    __device__ __forceinline__ void store(float* red, int g, int t) {
        red[g * 8 + 2 * t] = d[0];
        red[g * 8 + 2 * t + 1] = d[1];
        red[(g + 8) * 8 + 2 * t] = d[2];
        red[(g + 8) * 8 + 2 * t + 1] = d[3];
    }
};
template <>
struct GemvAcc<float> {
    float a[2][8];
    __device__ __forceinline__ void zero() {
#pragma unroll
        for (int m = 0; m < 8; ++m) a[0][m] = a[1][m] = 0.f;
    }
    __device__ __forceinline__ void step(const uint4& w0, const uint4& w1, const uint4* xs, int Mp, int M, int g) {
        float p[4], q[4], x[4];
        lb_unpack_chunk<float>(w0, p);
        lb_unpack_chunk<float>(w1, q);
#pragma unroll
        for (int m = 0; m < 8; ++m) {
            if (m >= M) break;
            lb_unpack_chunk<float>(xs[m], x);
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                a[0][m] = fmaf(p[i], x[i], a[0][m]);
                a[1][m] = fmaf(q[i], x[i], a[1][m]);
            }
        }
    }
    __device__ __forceinline__ void store(float* red, int g, int t) {
#pragma unroll
        for (int m = 0; m < 8; ++m)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                float v = a[h][m];
                v += __shfl_xor_sync(0xffffffffu, v, 1);
                v += __shfl_xor_sync(0xffffffffu, v, 2);
                if (t == 0) red[(g + 8 * h) * 8 + m] = v;
            }
    }
};

// the token columns of a chunk when they live in global memory as rows (routed experts, second product)
template <typename WT>
__device__ __forceinline__ void step_pairs(GemvAcc<WT>& acc, const uint4& w0, const uint4& w1, const uint8_t* pairs, size_t row_bytes,
                                           const int* pair, int chunk, int M, int g);
template <>
__device__ __forceinline__ void step_pairs<__nv_bfloat16>(GemvAcc<__nv_bfloat16>& acc, const uint4& w0, const uint4& w1, const uint8_t* pairs,
                                                          size_t row_bytes, const int* pair, int chunk, int M, int g) {
    const int pr = g < M ? pair[g] : -1;
    uint4 x = make_uint4(0, 0, 0, 0);
    if (pr >= 0) x = *reinterpret_cast<const uint4*>(pairs + (size_t)pr * row_bytes + (size_t)chunk * 16);
    mma_bf16(acc.d, w0.x, w1.x, w0.y, w1.y, x.x, x.y);
    mma_bf16(acc.d, w0.z, w1.z, w0.w, w1.w, x.z, x.w);
}
template <>
__device__ __forceinline__ void step_pairs<float>(GemvAcc<float>& acc, const uint4& w0, const uint4& w1, const uint8_t* pairs, size_t row_bytes,
                                                  const int* pair, int chunk, int M, int g) {
    float p[4], q[4], x[4];
    lb_unpack_chunk<float>(w0, p);
    lb_unpack_chunk<float>(w1, q);
#pragma unroll
    for (int m = 0; m < 8; ++m) {
        if (m >= M) break;
        const int pr = pair[m];
        if (pr < 0) continue;
        lb_unpack_chunk<float>(*reinterpret_cast<const uint4*>(pairs + (size_t)pr * row_bytes + (size_t)chunk * 16), x);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            acc.a[0][m] = fmaf(p[i], x[i], acc.a[0][m]);
            acc.a[1][m] = fmaf(q[i], x[i], acc.a[1][m]);
        }
    }
}

template <int NB>
struct GemvBatch {
    uint4 a[NB][2], b[NB][2];  // [slice][chunk t / t+4], rows g / g+8
};

// loads NB K slices (first, first + stride, ...; those below n) of a 16-row strip: lane (g, t) takes chunks t, t+4 of rows g, g+8
template <int NB>
__device__ __forceinline__ void load_batch(GemvBatch<NB>& w, const uint8_t* strip, int first, int stride, int n, int g, int t) {
#pragma unroll
    for (int u = 0; u < NB; ++u) {
        const int s = first + u * stride;
        if (s < n) {
            const uint8_t* p = strip + (size_t)s * kImgBlock + (size_t)t * 128 + (size_t)g * 16;
            w.a[u][0] = ldg_stream(p);
            w.a[u][1] = ldg_stream(p + 512);
            w.b[u][0] = ldg_stream(p + 1024);
            w.b[u][1] = ldg_stream(p + 1536);
        }
    }
}

// KW warps share a strip of 16 rows by K slices, 8/KW strips run side by side in a CTA.
template <typename WT, int PRO, int EPI>
__global__ void __launch_bounds__(kGemvThreads, 2) lb_dense_gemv_kernel(const LbDenseGemv p, int Mp_launch, int KW, bool vec) {
    extern __shared__ __align__(16) uint8_t smem[];
    constexpr int C = LbElem<WT>::kChunk;
    constexpr bool kDual = EPI == LB_DEPI_GLU || EPI == LB_DEPI_SILU;
    constexpr int NB = kDual ? 1 : 2;
    __shared__ float red[kGemvWarps][128];
    __shared__ float red2[kDual ? kGemvWarps : 1][128];
    __shared__ float s_stat[kGemvWarps];
    __shared__ int s_pair[kMaxLanesPerPass], s_tok[kMaxLanesPerPass], s_n;
    __shared__ float s_w[kMaxLanesPerPass];
    constexpr bool kStage = EPI == LB_DEPI_STAGE;
    // columns of this CTA: every token; the token of a staging CTA; the tokens that chose this CTA's expert
    int M = kStage ? 1 : p.M, Mp = kStage ? 1 : Mp_launch;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int SP = kGemvWarps / KW, kw = warp % KW, sp = warp / KW;
    const int strips = lb_ceil_div(p.rows, 16), chunks = p.slices * 8;
    uint4* xs = reinterpret_cast<uint4*>(smem);  // [chunk][Mp]
    const uint8_t *w1 = p.w, *w2 = p.w2;

    // the weights do not depend on earlier launches: the first batch is requested before the dependency wait
    GemvBatch<NB> cur, cur2;
    int strip = (int)blockIdx.x * SP + sp;
    auto strip_ptr = [&](const uint8_t* base, int st) { return base + (size_t)(st >> 3) * p.slices * kImgBlock + (size_t)(st & 7) * 2048; };
    constexpr bool kEarly = PRO != LB_DPRO_MOE && PRO != LB_DPRO_PAIRS && !kStage;
    if (kEarly && strip < strips) {
        load_batch(cur, strip_ptr(w1, strip), kw, KW, p.slices, g, t);
        if (kDual) load_batch(cur2, strip_ptr(w2, strip), kw, KW, p.slices, g, t);
    }
    lb_pdl_launch_dependents();
    lb_pdl_wait();

    if (PRO == LB_DPRO_MOE) {
        // every CTA repeats the choice of experts: a warp per token, `top` rounds of a warp-wide first maximum
        float* sl = reinterpret_cast<float*>(smem + (size_t)chunks * Mp * 16);  // [M][experts]
        int* s_idx = reinterpret_cast<int*>(sl + (size_t)p.M * p.experts);     // [M][top]
        if (warp < p.M) {
            float* row = sl + (size_t)warp * p.experts;
            for (int e = lane; e < p.experts; e += 32) row[e] = p.logits[(size_t)warp * p.ldl + e];
            __syncwarp();
            for (int j = 0; j < p.top; ++j) {
                float best = -INFINITY;
                int bi = 0x7fffffff;
                for (int e = lane; e < p.experts; e += 32)
                    if (row[e] > best) {
                        best = row[e];
                        bi = e;
                    }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
                    const float ov = __shfl_xor_sync(0xffffffffu, best, o);
                    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
                    if (ov > best || (ov == best && oi < bi)) {
                        best = ov;
                        bi = oi;
                    }
                }
                if (bi >= p.experts) bi = 0;  // only NaNs left
                if (lane == 0) {
                    s_idx[warp * p.top + j] = bi;
                    row[bi] = -INFINITY;
                }
                __syncwarp();
            }
        }
        __syncthreads();
        const int pairs = p.M * p.top;
        auto first_of = [&](int pr) {  // whether this (token, choice) is the first that names its expert
            for (int q = 0; q < pr; ++q)
                if (s_idx[q] == s_idx[pr]) return false;
            return true;
        };
        if (blockIdx.x == 0 && blockIdx.y == 0 && tid < pairs && first_of(tid)) {
            int at = 0;
            for (int q = 0; q < tid; ++q) at += first_of(q) ? 1 : 0;
            p.list->expert[at] = s_idx[tid];
            for (int m = 0; m < p.M; ++m) {
                int found = -1;
                for (int j = 0; j < p.top; ++j)
                    if (s_idx[m * p.top + j] == s_idx[tid]) found = m * p.top + j;
                p.list->pair[at][m] = found;
            }
        }
        if (blockIdx.x == 0 && blockIdx.y == 0 && tid == 0) {
            int n = 0;
            for (int q = 0; q < pairs; ++q) n += first_of(q) ? 1 : 0;
            p.list->n = n;
        }
        const int mine = blockIdx.y;
        if (!first_of(mine)) return;  // uniform over the CTA
        const int e = s_idx[mine];
        w1 += (size_t)e * p.group_bytes;
        w2 += (size_t)e * p.group_bytes;
        if (tid == 0) {
            int n = 0;
            for (int q = 0; q < pairs; ++q)
                if (s_idx[q] == e) {
                    s_pair[n] = q;
                    s_tok[n] = q / p.top;
                    s_w[n] = lb_sigmoidf(p.logits[(size_t)(q / p.top) * p.ldl + e]);
                    ++n;
                }
            s_n = n;
        }
        if (strip < strips) {
            load_batch(cur, strip_ptr(w1, strip), kw, KW, p.slices, g, t);
            load_batch(cur2, strip_ptr(w2, strip), kw, KW, p.slices, g, t);
        }
        __syncthreads();
        M = s_n;
        Mp = 1;
        while (Mp < M) Mp *= 2;
    }

    if (PRO == LB_DPRO_STAGED) {
        for (int i = tid; i < chunks * Mp; i += kGemvThreads) xs[i] = p.staged[i];
        __syncthreads();
    } else if (PRO != LB_DPRO_PAIRS) {
        // ---- input rows: 8/Mp warps per token ----
        const int WPT = kGemvWarps / Mp, m = warp / WPT, wt = warp % WPT, lt = wt * 32 + lane, nt = WPT * 32;
        const bool live = m < M;
        const int tok = !live ? 0 : kStage ? (int)blockIdx.x : PRO == LB_DPRO_MOE ? s_tok[m] : m;
        const int src = p.row_idx ? p.row_idx[tok] : tok;
        const float* xr = p.x + (size_t)src * p.ldx;
        float rstd = 0.f, gain = 1.f;
        float* s_head = nullptr;
        int heads = 0;
        if (PRO == LB_DPRO_NORM || PRO == LB_DPRO_CONV || PRO == LB_DPRO_MOE) {
            float ss = 0.f;
            if (live)
                for (int k = lt; k < p.K; k += nt) ss = fmaf(xr[k], xr[k], ss);
            ss = lb_warp_sumf(ss);
            if (lane == 0) s_stat[warp] = ss;
            __syncthreads();
            float tot = 0.f;
            for (int i = 0; i < WPT; ++i) tot += s_stat[m * WPT + i];
            rstd = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(tot, (float)p.K), p.eps)));
            if (p.gain) gain = *p.gain;
        }
        if (PRO == LB_DPRO_GATED) {
            heads = p.K / p.head_dim;
            s_head = reinterpret_cast<float*>(smem + (size_t)chunks * Mp * 16) + (size_t)m * heads;
            if (live)
                for (int h = wt; h < heads; h += WPT) {
                    float ss = 0.f;
                    for (int i = lane; i < p.head_dim; i += 32) {
                        const float v = xr[h * p.head_dim + i];
                        ss = fmaf(v, v, ss);
                    }
                    ss = lb_warp_sumf(ss);
                    if (lane == 0) s_head[h] = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.head_dim), p.eps)));
                }
            __syncthreads();
        }
        const int seq = p.lane0 + tok;
        int pos = 0;
        if (PRO == LB_DPRO_CONV && live) pos = p.pos[tok];
        for (int c = lt; c < chunks; c += nt) {
            float f[C];
            const int k0 = c * C;
            if (live && k0 < p.K) {
                lb_load_cols<C>(xr, k0, p.K, vec, f);
                if (PRO == LB_DPRO_NORM || PRO == LB_DPRO_CONV || PRO == LB_DPRO_MOE) {
#pragma unroll
                    for (int i = 0; i < C; ++i) f[i] = f[i] * rstd * gain;
                    if (p.gain_w) {
                        float w[C];
                        lb_load_cols<C>(p.gain_w, k0, p.K, vec, w);
#pragma unroll
                        for (int i = 0; i < C; ++i) f[i] *= w[i];
                    }
                    if (PRO == LB_DPRO_NORM && p.x_out && (kStage || blockIdx.x == 0)) {
#pragma unroll
                        for (int i = 0; i < C; ++i)
                            if (k0 + i < p.K) p.x_out[(size_t)tok * p.ldx + k0 + i] = f[i];
                    }
                }
                if (PRO == LB_DPRO_MOE) {
#pragma unroll
                    for (int i = 0; i < C; ++i) f[i] *= s_w[m];
                }
                if (PRO == LB_DPRO_GATED) {
                    float gt[C], hw[C];
                    lb_load_cols<C>(p.gate + (size_t)tok * p.gate_ld, k0, p.K, vec, gt);
                    lb_load_cols<C>(p.head_w, k0, p.K, vec, hw);
#pragma unroll
                    for (int i = 0; i < C; ++i) {
                        const int k = k0 + i, h = k / p.head_dim;
                        if (k < p.K) f[i] = f[i] * s_head[h] * hw[i] * (p.gate_sigmoid ? lb_sigmoidf(gt[i]) : lb_siluf(gt[i]));
                    }
                }
                if (PRO == LB_DPRO_CONV) {
                    float* ring = p.conv_ring + (size_t)seq * p.taps * p.ring_ld;
                    float a[C], w[C], y[C];
#pragma unroll
                    for (int i = 0; i < C; ++i) a[i] = 0.f;
                    for (int j = 0; j + 1 < p.taps; ++j) {  // tap j looks back taps - 1 - j positions
                        const int ps = pos - (p.taps - 1) + j;
                        if (ps < 0) continue;
                        lb_load_cols<C>(p.conv_w + (size_t)j * p.ring_ld, k0, p.K, vec, w);
                        lb_load_cols<C>(ring + (size_t)(ps % p.taps) * p.ring_ld, k0, p.K, vec, y);
#pragma unroll
                        for (int i = 0; i < C; ++i) a[i] = fmaf(w[i], y[i], a[i]);
                    }
                    lb_load_cols<C>(p.conv_w + (size_t)(p.taps - 1) * p.ring_ld, k0, p.K, vec, w);
                    float* slot = ring + (size_t)(pos % p.taps) * p.ring_ld + k0;  // no CTA of this launch reads this slot
#pragma unroll
                    for (int i = 0; i < C; ++i) {
                        a[i] = fmaf(w[i], f[i], a[i]);
                        if ((kStage || blockIdx.x == 0) && k0 + i < p.K) slot[i] = f[i];
                        f[i] += a[i];
                    }
                }
            } else {
#pragma unroll
                for (int i = 0; i < C; ++i) f[i] = 0.f;
            }
            if (kStage) {
                p.staged[(size_t)c * Mp_launch + tok] = lb_pack_chunk<WT>(f);
                continue;
            }
            xs[(size_t)c * Mp + m] = lb_pack_chunk<WT>(f);
        }
        __syncthreads();
    }

    if (kStage) return;

    const int nact = PRO == LB_DPRO_PAIRS ? p.list->n : 1;

    for (; strip - sp < strips; strip += (int)gridDim.x * SP) {
        GemvAcc<WT> acc, acc2;
        acc.zero();
        if (kDual) acc2.zero();
        if (strip < strips) {
            if (PRO != LB_DPRO_PAIRS) {
                const uint8_t* s1 = strip_ptr(w1, strip);
                const uint8_t* s2 = kDual ? strip_ptr(w2, strip) : nullptr;
                const int next = strip + (int)gridDim.x * SP;
                for (int s = kw; s < p.slices; s += NB * KW) {
                    GemvBatch<NB> now = cur, now2;
                    if (kDual) now2 = cur2;
                    if (s + NB * KW < p.slices) {
                        load_batch(cur, s1, s + NB * KW, KW, p.slices, g, t);
                        if (kDual) load_batch(cur2, s2, s + NB * KW, KW, p.slices, g, t);
                    } else if (next < strips) {  // the next strip's first batch travels while this strip's sums meet
                        load_batch(cur, strip_ptr(w1, next), kw, KW, p.slices, g, t);
                        if (kDual) load_batch(cur2, strip_ptr(w2, next), kw, KW, p.slices, g, t);
                    }
#pragma unroll
                    for (int u = 0; u < NB; ++u) {
                        const int sl = s + u * KW;
                        if (sl < p.slices) {
                            const uint4* x0 = xs + (size_t)(sl * 8 + t) * Mp;
                            acc.step(now.a[u][0], now.b[u][0], x0, Mp, M, g);
                            acc.step(now.a[u][1], now.b[u][1], x0 + 4 * Mp, Mp, M, g);
                            if (kDual) {
                                acc2.step(now2.a[u][0], now2.b[u][0], x0, Mp, M, g);
                                acc2.step(now2.a[u][1], now2.b[u][1], x0 + 4 * Mp, Mp, M, g);
                            }
                        }
                    }
                }
            } else {
                // K runs over the experts of the list one after the other
                const int total = nact * p.slices;
                const size_t row_bytes = (size_t)p.ldp * sizeof(WT);
                for (int s = kw; s < total; s += 4 * KW) {
                    uint4 wa[4][2], wb[4][2];
                    int at[4], sl[4];
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        const int i = s + u * KW < total ? s + u * KW : s;
                        at[u] = i / p.slices;
                        sl[u] = i - at[u] * p.slices;
                        const uint8_t* q = strip_ptr(w1 + (size_t)p.list->expert[at[u]] * p.group_bytes, strip) + (size_t)sl[u] * kImgBlock + (size_t)t * 128 + (size_t)g * 16;
                        wa[u][0] = ldg_stream(q);
                        wa[u][1] = ldg_stream(q + 512);
                        wb[u][0] = ldg_stream(q + 1024);
                        wb[u][1] = ldg_stream(q + 1536);
                    }
#pragma unroll
                    for (int u = 0; u < 4; ++u) {
                        if (s + u * KW >= total) break;
                        step_pairs<WT>(acc, wa[u][0], wb[u][0], p.pairs, row_bytes, p.list->pair[at[u]], sl[u] * 8 + t, p.M, g);
                        step_pairs<WT>(acc, wa[u][1], wb[u][1], p.pairs, row_bytes, p.list->pair[at[u]], sl[u] * 8 + t + 4, p.M, g);
                    }
                }
            }
        }
        __syncthreads();  // the previous strip's sums are no longer read
        acc.store(red[warp], g, t);
        if (kDual) acc2.store(red2[warp], g, t);
        __syncthreads();
        for (int o = tid; o < SP * 128; o += kGemvThreads) {
            const int s = o >> 7, e = o & 127, r = e >> 3, m = e & 7;
            const int row = (strip - sp + s) * 16 + r;
            if (m >= M || row >= p.rows) continue;
            float v = 0.f, u = 0.f;
            for (int k = 0; k < KW; ++k) {
                v += red[s * KW + k][e];
                if (kDual) u += red2[s * KW + k][e];
            }
            if (EPI == LB_DEPI_F32) p.out[(size_t)m * p.ldo + row] = v;
            if (EPI == LB_DEPI_RESID) {
                const size_t at = (size_t)m * p.ldo + row;
                p.out[at] = fmaf(p.mult, v, p.res_mult * (p.res ? p.res : p.out)[at]);
            }
            if (EPI == LB_DEPI_GELU) p.out[(size_t)m * p.ldo + row] = lb_gelu_erff(v);
            if (EPI == LB_DEPI_SILU) p.out[(size_t)m * p.ldo + row] = lb_siluf(v) * u;
            if (EPI == LB_DEPI_GLU) {
                reinterpret_cast<WT*>(p.out_pairs)[(size_t)s_pair[m] * p.ldo + row] = (WT)lb_clamped_glu(v, u, p.limit);
            }
        }
    }
}

constexpr int kStageTokens = 3;  // from this many tokens on the input rows are made once, by a launch of their own

template <typename WT, int PRO, int EPI>
int gemv_launch(loom_b200_ctx* ctx, const LbDenseGemv& pin) {
    LbDenseGemv p = pin;
    LB_REQUIRE(ctx, p.M >= 1 && p.M <= kMaxLanesPerPass, "dense_gemv: %d tokens", p.M);
    int Mp = 1;
    while (Mp < p.M) Mp *= 2;
    const int strips = lb_ceil_div(p.rows, 16), cap = ctx->sm_count * 2;
    int KW = 1;
    while (KW < kGemvWarps && KW * 2 <= p.slices) KW *= 2;
    // many strips per CTA: fewer warps per strip, so that a warp streams longer runs between two meetings of the sums
    while (KW > 1 && (long long)strips >= 6ll * (2 * kGemvWarps / KW) * cap) KW /= 2;
    const int SP = kGemvWarps / KW;
    bool vec = PRO == LB_DPRO_STAGED || PRO == LB_DPRO_PAIRS || lb_vec_rows(p.x, p.ldx);
    if (PRO == LB_DPRO_GATED) vec = vec && lb_vec_rows(p.gate, p.gate_ld) && lb_vec_rows(p.head_w, 4);
    if (p.gain_w) vec = vec && lb_vec_rows(p.gain_w, 4);
    if (PRO == LB_DPRO_CONV) vec = vec && lb_vec_rows(p.conv_w, p.ring_ld) && lb_vec_rows(p.conv_ring, p.ring_ld);
    const size_t rows_smem = (size_t)p.slices * 8 * (EPI == LB_DEPI_STAGE ? 1 : Mp) * 16;
    size_t smem = PRO == LB_DPRO_PAIRS || EPI == LB_DEPI_STAGE ? 0 : rows_smem;
    if (PRO == LB_DPRO_MOE) smem += (size_t)p.M * p.experts * 4 + (size_t)p.M * p.top * 4;
    if (PRO == LB_DPRO_GATED) smem = rows_smem + (size_t)Mp * (p.K / p.head_dim) * 4;
    if (smem > kGemvSmemX + 16 * 1024) return lb_fail(ctx, LOOM_B200_ERR_UNSUPPORTED, "dense_gemv: %d tokens of %d columns need %zu B of shared memory", p.M, p.K, smem);
    if (smem > 48 * 1024) LB_BIG_SMEM(ctx, (lb_dense_gemv_kernel<WT, PRO, EPI>), kGemvSmemX + 16 * 1024);
    int gx = lb_ceil_div(strips, SP), gy = 1, share = cap;
    if (EPI == LB_DEPI_STAGE) {
        gx = share = p.M;
    } else if (PRO == LB_DPRO_MOE) {
        gy = p.M * p.top;
        share = cap / (gy < p.experts ? gy : p.experts);
        if (share < 1) share = 1;
    }
    if (gx > share) gx = lb_ceil_div(gx, lb_ceil_div(gx, share));  // equal numbers of strips per CTA
    LB_LAUNCH(ctx, (lb_dense_gemv_kernel<WT, PRO, EPI>), dim3(gx, gy), dim3(kGemvThreads), smem, p, Mp, KW, vec);
    return 0;
}

// a product whose input rows take some work: inside every CTA for one or two tokens, as a launch of their own for more
template <typename WT, int PRO, int EPI>
int gemv_rows(loom_b200_ctx* ctx, const LbDenseGemv& pin) {
    if (pin.M < kStageTokens) return gemv_launch<WT, PRO, EPI>(ctx, pin);
    LbDenseGemv p = pin;
    const size_t bytes = (size_t)p.slices * 8 * kMaxLanesPerPass * 16;
    if (bytes > ctx->stage_scratch_bytes) {
        if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "the staging buffer of the GEMV would grow while recording a graph");
        LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        if (ctx->stage_scratch) cudaFree(ctx->stage_scratch);
        ctx->stage_scratch = nullptr;
        ctx->stage_scratch_bytes = 0;
        LB_CUDA(ctx, cudaMalloc(&ctx->stage_scratch, bytes));
        ctx->stage_scratch_bytes = bytes;
    }
    p.staged = static_cast<uint4*>(ctx->stage_scratch);
    if (int rc = gemv_launch<WT, PRO, LB_DEPI_STAGE>(ctx, p)) return rc;
    return gemv_launch<WT, LB_DPRO_STAGED, EPI>(ctx, p);
}

template <typename WT>
int gemv_dispatch(loom_b200_ctx* ctx, int pro, int epi, const LbDenseGemv& p) {
#define LB_CASE(P, E, RUN) \
    if (pro == P && epi == E) return RUN<WT, P, E>(ctx, p)
    LB_CASE(LB_DPRO_CONV, LB_DEPI_F32, gemv_rows);
    LB_CASE(LB_DPRO_NORM, LB_DEPI_F32, gemv_rows);
    LB_CASE(LB_DPRO_NORM, LB_DEPI_GELU, gemv_rows);
    LB_CASE(LB_DPRO_NORM, LB_DEPI_SILU, gemv_rows);
    LB_CASE(LB_DPRO_PLAIN, LB_DEPI_F32, gemv_launch);
    LB_CASE(LB_DPRO_PLAIN, LB_DEPI_RESID, gemv_launch);
    LB_CASE(LB_DPRO_GATED, LB_DEPI_RESID, gemv_rows);
    LB_CASE(LB_DPRO_MOE, LB_DEPI_GLU, gemv_launch);
    LB_CASE(LB_DPRO_PAIRS, LB_DEPI_RESID, gemv_launch);
#undef LB_CASE
    return lb_fail(ctx, LOOM_B200_ERR_UNSUPPORTED, "dense_gemv: prologue %d with epilogue %d is not built", pro, epi);
}

// ---- token-block GEMM with plain fused multiply-adds (32-bit floats) -------------------------------------------

constexpr int kSimtTile = 64;

template <typename WT, int EPI>
__global__ void __launch_bounds__(256) lb_dense_gemm_simt_kernel(const LbDenseGemm p) {
    constexpr int C = LbElem<WT>::kChunk;
    constexpr bool kDual = EPI == LB_DEPI_GLU || EPI == LB_DEPI_SILU;
    __shared__ __align__(16) uint8_t sa[8192], sb[8192], sb2[kDual ? 8192 : 16];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int tid = threadIdx.x, tl = tid & 31, rg = tid >> 5;
    const int row0 = blockIdx.x * kSimtTile, tok0 = blockIdx.y * kSimtTile;
    const uint8_t *w = p.w, *w2 = p.w2;
    if (p.nblocks) {
        if (tok0 / kImgRows >= *p.nblocks) return;
        const size_t off = (size_t)p.block_group[tok0 / kImgRows] * p.group_bytes;
        w += off;
        w2 += kDual ? off : 0;
    }
    float acc[2][8], acc2[2][8];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[i][j] = acc2[i][j] = 0.f;
    const size_t abase = (size_t)(tok0 >> 7) * p.slices * kImgBlock + (size_t)((tok0 & 127) >> 3) * 1024;
    const size_t bbase = (size_t)(row0 >> 7) * p.slices * kImgBlock + (size_t)((row0 & 127) >> 3) * 1024;
    for (int s = 0; s < p.slices; ++s) {
        __syncthreads();
        for (int i = tid; i < 512; i += 256) {
            reinterpret_cast<uint4*>(sa)[i] = *reinterpret_cast<const uint4*>(p.x + abase + (size_t)s * kImgBlock + (size_t)i * 16);
            reinterpret_cast<uint4*>(sb)[i] = *reinterpret_cast<const uint4*>(w + bbase + (size_t)s * kImgBlock + (size_t)i * 16);
            if (kDual) reinterpret_cast<uint4*>(sb2)[i] = *reinterpret_cast<const uint4*>(w2 + bbase + (size_t)s * kImgBlock + (size_t)i * 16);
        }
        __syncthreads();
        for (int c = 0; c < 8; ++c) {
            float a0[C], a1[C], b[C];
            lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(sa + (tl >> 3) * 1024 + c * 128 + (tl & 7) * 16), a0);
            lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(sa + ((tl >> 3) + 4) * 1024 + c * 128 + (tl & 7) * 16), a1);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(sb + rg * 1024 + c * 128 + j * 16), b);
#pragma unroll
                for (int i = 0; i < C; ++i) {
                    acc[0][j] = fmaf(a0[i], b[i], acc[0][j]);
                    acc[1][j] = fmaf(a1[i], b[i], acc[1][j]);
                }
                if (kDual) {
                    lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(sb2 + rg * 1024 + c * 128 + j * 16), b);
#pragma unroll
                    for (int i = 0; i < C; ++i) {
                        acc2[0][j] = fmaf(a0[i], b[i], acc2[0][j]);
                        acc2[1][j] = fmaf(a1[i], b[i], acc2[1][j]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int tok = tok0 + tl + 32 * i, r = row0 + rg * 8;
        if (!p.nblocks && tok >= p.tokens) continue;
        if (EPI == LB_DEPI_F32 || EPI == LB_DEPI_RESID) {
            if (r >= p.ldo) continue;
            float* o = p.out + (size_t)tok * p.ldo + r;
#pragma unroll
            for (int j = 0; j < 8; ++j) o[j] = EPI == LB_DEPI_F32 ? acc[i][j] : fmaf(p.mult, acc[i][j], p.res_mult * o[j]);
        } else {
            float f[8];
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                f[j] = acc[i][j];
                if (EPI == LB_DEPI_GELU) f[j] = lb_gelu_erff(acc[i][j]);
                if (EPI == LB_DEPI_GLU) f[j] = lb_clamped_glu(acc[i][j], acc2[i][j], p.limit);
                if (EPI == LB_DEPI_SILU) f[j] = lb_siluf(acc[i][j]) * acc2[i][j];
            }
            if (EPI == LB_DEPI_HEADS) {
                if (r < p.rows) *reinterpret_cast<uint4*>(p.img + lb_heads_chunk(tok, r, p.heads, p.head_dim, p.head_chunks)) = lb_pack_chunk<__nv_bfloat16>(f);
            } else if (r / LbElem<WT>::kSlice < p.img_slices) {
                lb_img_store8<WT>(p.img, tok, r, p.img_slices, f);
            }
        }
    }
}

template <typename WT>
int gemm_simt(loom_b200_ctx* ctx, int epi, const LbDenseGemm& p) {
    // rows: every 64-row tile that holds a row or a column of the output image's padding
    const int rows = lb_round_up(p.rows, kSimtTile);
    const int blocks = p.nblocks ? p.max_blocks * 2 : lb_ceil_div(p.tokens, kSimtTile);
    const dim3 grid(rows / kSimtTile, blocks);
#define LB_CASE(E)                                                                           \
    if (epi == E) {                                                                          \
        LB_LAUNCH(ctx, (lb_dense_gemm_simt_kernel<WT, E>), grid, dim3(256), 0, p);           \
        return 0;                                                                            \
    }
    LB_CASE(LB_DEPI_F32)
    LB_CASE(LB_DEPI_RESID)
    LB_CASE(LB_DEPI_GELU)
    LB_CASE(LB_DEPI_GLU)
    LB_CASE(LB_DEPI_SILU)
    LB_CASE(LB_DEPI_IMG)
    LB_CASE(LB_DEPI_HEADS)
#undef LB_CASE
    return lb_fail(ctx, LOOM_B200_ERR_UNSUPPORTED, "dense_gemm: epilogue %d is not built", epi);
}

}  // namespace

int lb_gemm_bf16_run(loom_b200_ctx* ctx, int epi, const LbDenseGemm& p);  // gemm_bf16.cu

int lb_dense_gemv_max_tokens(int K, int dtype) {
    const size_t row = (size_t)lb_slices_of(K, dtype) * 128;
    int m = kMaxLanesPerPass;
    while (m > 1 && (size_t)m * row > kGemvSmemX) m /= 2;
    return m;
}

int lb_dense_gemv(loom_b200_ctx* ctx, int dtype, int pro, int epi, const LbDenseGemv& p) {
    return dtype == LOOM_B200_DTYPE_BF16 ? gemv_dispatch<__nv_bfloat16>(ctx, pro, epi, p) : gemv_dispatch<float>(ctx, pro, epi, p);
}

int lb_dense_gemm(loom_b200_ctx* ctx, int dtype, int epi, const LbDenseGemm& pin) {
    LbDenseGemm p = pin;
    p.status = ctx->status_dev;
    LB_REQUIRE(ctx, p.x && p.w && p.rows > 0 && p.slices > 0 && (p.tokens > 0 || p.nblocks), "dense_gemm: bad arguments");
    LB_REQUIRE(ctx, (epi != LB_DEPI_F32 && epi != LB_DEPI_RESID) || p.ldo % 8 == 0, "dense_gemm: output rows of %d floats", p.ldo);
    if (dtype == LOOM_B200_DTYPE_F32) return gemm_simt<float>(ctx, epi, p);
    if (!ctx->opt_dense_tc) return gemm_simt<__nv_bfloat16>(ctx, epi, p);
    return lb_gemm_bf16_run(ctx, epi, p);
}

extern "C" {

int loom_b200_matrix_create(loom_b200_ctx* ctx, int rows, int cols, int groups, int dtype, loom_b200_matrix** out) {
    if (!ctx) return lb_fail(nullptr, LOOM_B200_ERR_INVALID, "matrix_create: ctx is NULL");
    LB_REQUIRE(ctx, out != nullptr, "matrix_create: out is NULL");
    *out = nullptr;
    LB_REQUIRE(ctx, rows > 0 && cols > 0 && groups > 0, "matrix_create: bad shape %dx%d (%d groups)", rows, cols, groups);
    LB_REQUIRE(ctx, dtype == LOOM_B200_DTYPE_F32 || dtype == LOOM_B200_DTYPE_BF16, "matrix_create: dtype %d", dtype);
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "matrix_create cannot be recorded");
    if (int rc = lb_set_device(ctx)) return rc;
    auto* m = new loom_b200_matrix();
    m->rows = rows;
    m->cols = cols;
    m->groups = groups;
    m->dtype = dtype;
    m->slices = lb_slices_of(cols, dtype);
    m->group_bytes = lb_img_bytes(rows, cols, dtype);
    m->device = ctx->device;
    const size_t bytes = m->group_bytes * groups;
    cudaError_t e = cudaMalloc(&m->data, bytes);
    if (e == cudaSuccess) e = cudaMemsetAsync(m->data, 0, bytes, ctx->stream);
    if (e != cudaSuccess) {
        if (m->data) cudaFree(m->data);
        delete m;
        return lb_fail(ctx, LOOM_B200_ERR_CUDA, "matrix_create: %zu bytes: %s", bytes, cudaGetErrorString(e));
    }
    *out = m;
    return 0;
}

int loom_b200_matrix_put(loom_b200_ctx* ctx, loom_b200_matrix* m, int group, int row0, int rows, const void* src, int src_dtype, int src_on_device) {
    if (!ctx) return lb_fail(nullptr, LOOM_B200_ERR_INVALID, "matrix_put: ctx is NULL");
    LB_REQUIRE(ctx, m && src, "matrix_put: NULL argument");
    LB_REQUIRE(ctx, group >= 0 && group < m->groups && row0 >= 0 && rows > 0 && row0 + rows <= m->rows, "matrix_put: rows %d..%d of group %d in %dx%d (%d groups)",
               row0, row0 + rows, group, m->rows, m->cols, m->groups);
    LB_REQUIRE(ctx, src_dtype == LOOM_B200_DTYPE_F32 || src_dtype == LOOM_B200_DTYPE_BF16, "matrix_put: dtype %d", src_dtype);
    LB_REQUIRE(ctx, m->device == ctx->device, "matrix_put: matrix lives on device %d", m->device);
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "matrix_put cannot be recorded");
    if (int rc = lb_set_device(ctx)) return rc;
    const size_t bytes = (size_t)rows * m->cols * (src_dtype == LOOM_B200_DTYPE_BF16 ? 2 : 4);
    const void* dev = src;
    if (!src_on_device) {
        if (int rc = lb_ensure_scratch(ctx, bytes)) return rc;
        LB_CUDA(ctx, cudaMemcpyAsync(ctx->scratch, src, bytes, cudaMemcpyHostToDevice, ctx->stream));
        dev = ctx->scratch;
    }
    const size_t threads = (size_t)rows * m->slices * 8;
    const unsigned grid = (unsigned)((threads + 255) / 256);
    uint8_t* img = m->data + (size_t)group * m->group_bytes;
    if (m->dtype == LOOM_B200_DTYPE_BF16)
        lb_image_put_kernel<__nv_bfloat16><<<grid, 256, 0, ctx->stream>>>(dev, src_dtype, rows, m->cols, row0, m->slices, img);
    else
        lb_image_put_kernel<float><<<grid, 256, 0, ctx->stream>>>(dev, src_dtype, rows, m->cols, row0, m->slices, img);
    LB_CHECK_LAUNCH(ctx, "lb_image_put_kernel");
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    return 0;
}

int loom_b200_matrix_info(const loom_b200_matrix* m, int* rows, int* cols, int* groups, int* dtype) {
    if (!m) return lb_fail(nullptr, LOOM_B200_ERR_INVALID, "matrix_info: matrix is NULL");
    if (rows) *rows = m->rows;
    if (cols) *cols = m->cols;
    if (groups) *groups = m->groups;
    if (dtype) *dtype = m->dtype;
    return 0;
}

void loom_b200_matrix_free(loom_b200_ctx* ctx, loom_b200_matrix* m) {
    if (!m) return;
    if (ctx) {
        cudaSetDevice(ctx->device);
        cudaStreamSynchronize(ctx->stream);
    }
    if (m->data) cudaFree(m->data);
    delete m;
}

}  // extern "C"
