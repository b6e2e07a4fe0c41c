// delta_rule.cu -- gated delta rule with one decay per head behind short convolutions: the one-token step and the token block.
//
//   S' = g_t S_(t-1),  u_t = beta_t (v_t - S'^T k_t),  S_t = S' + k_t u_t^T,  o_t = S_t^T q_t
//
// A block of tokens is cut into chunks of C.  With G_t the product of the decays inside a chunk and S the state in front of it,
//   u_t + sum_(s < t) L_ts u_s = beta_t v_t - beta_t G_t S^T k_t,   L_ts = beta_t (G_t / G_s) k_t.k_s
// so (I + L)^-1 times (beta v | beta G k) gives u = Wv - Wk S without knowing S, and
//   o_t   = (G_t q_t - sum_s A_ts wk_s)^T S + sum_s A_ts wv_s,   A_ts = (G_t / G_s) q_t.k_s, s <= t
//   S_end = (G_C - Kd^T Wk) S + Kd^T Wv,                         Kd_s = (G_C / G_s) k_s
// Only the last line runs chunk after chunk.  Ratios of decays come from differences of their logarithms (no exponent is ever
// positive), summed in 64-bit so that a strong decay early in a chunk costs its later tokens nothing.  All the rest is 32-bit floats.
#include "mixers.cuh"

namespace {

constexpr int kMaxTaps = 16;
constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ float softplusf(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float log_gate(const LbDelta& p, const float* row, int h) {
    const int at = lb_delta_channels(p) + p.heads * p.vdim + p.heads + h;
    return -expf(p.a_log[h]) * softplusf(row[at] + p.dt_bias[h]);
}
__device__ __forceinline__ float write_strength(const LbDelta& p, const float* row, int h) {
    return lb_sigmoidf(row[lb_delta_channels(p) + p.heads * p.vdim + h]);
}

// ---- one token of each of M sequences: CTA = (32 value columns, head, sequence); warps split the key channels -----------
constexpr int kKeep = 16;  // state rows a thread keeps in registers

__global__ void __launch_bounds__(256) lb_delta_step_kernel(const LbDelta p, const int* pos_of, int lane0) {
    extern __shared__ float sm[];
    __shared__ float part[8][32], red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.y, m = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int hk = h / (p.heads / p.kv_heads), nch = lb_delta_channels(p), QK = p.kv_heads * p.dim, pos = pos_of[m];
    float *sq = sm, *sk = sm + p.dim;
    const float* row = p.proj + (size_t)m * p.ldp;
    float* ring = p.ring + (size_t)(lane0 + m) * p.taps * nch;
    const int v = blockIdx.x * 32 + lane;
    const bool live = v < p.vdim, fresh = pos == 0;
    float* S = p.state + (((size_t)(lane0 + m) * p.heads + h) * p.dim) * p.vdim + v;
    float old[kKeep];
#pragma unroll
    for (int i = 0; i < kKeep; ++i) {
        const int d = warp + 8 * i;
        old[i] = live && !fresh && d < p.dim ? S[(size_t)d * p.vdim] : 0.f;
    }
    // the convolution of one channel; `keep`: this thread puts the channel's projection into the ring (no CTA reads that slot now)
    auto conv = [&](int ch, bool keep) {
        const float x = row[ch];
        float a = 0.f;
        for (int j = 0; j + 1 < p.taps; ++j) {  // tap j looks back taps - 1 - j positions
            const int ps = pos - (p.taps - 1) + j;
            if (ps >= 0) a = fmaf(p.conv_w[(size_t)j * nch + ch], ring[(size_t)(ps % p.taps) * nch + ch], a);
        }
        a = fmaf(p.conv_w[(size_t)(p.taps - 1) * nch + ch], x, a);
        if (keep) ring[(size_t)(pos % p.taps) * nch + ch] = x;
        return lb_siluf(a);
    };
    const bool first = blockIdx.x == 0 && h % (p.heads / p.kv_heads) == 0;
    float qq = 0.f, kk = 0.f;
    for (int d = tid; d < p.dim; d += 256) {
        const float q = conv(hk * p.dim + d, first), k = conv(QK + hk * p.dim + d, first);
        sq[d] = q;
        sk[d] = k;
        qq = fmaf(q, q, qq);
        kk = fmaf(k, k, kk);
    }
    // (every warp convolves the CTA's value columns for itself; the first one keeps them)
    const float vv = live ? conv(2 * QK + h * p.vdim + v, warp == 0) : 0.f;
    const float beta = write_strength(p, row, h), g = expf(log_gate(p, row, h));
    qq = lb_block_sumf(qq, red);
    kk = lb_block_sumf(kk, red);
    const float rq = __fdiv_rn(p.qscale, sqrtf(qq + kUnitEps)), rk = __fdiv_rn(1.f, sqrtf(kk + kUnitEps));
    float a = 0.f;
    if (live) {
#pragma unroll
        for (int i = 0; i < kKeep; ++i)
            if (warp + 8 * i < p.dim) {
                old[i] *= g;
                a = fmaf(old[i], sk[warp + 8 * i] * rk, a);
            }
        for (int d = warp + 8 * kKeep; d < p.dim; d += 8) a = fmaf(fresh ? 0.f : g * S[(size_t)d * p.vdim], sk[d] * rk, a);
    }
    part[warp][lane] = a;
    __syncthreads();
    float sum = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sum += part[w][lane];
    const float u = beta * (vv - sum);
    a = 0.f;
    if (live) {
#pragma unroll
        for (int i = 0; i < kKeep; ++i) {
            const int d = warp + 8 * i;
            if (d < p.dim) {
                const float s = fmaf(sk[d] * rk, u, old[i]);
                S[(size_t)d * p.vdim] = s;
                a = fmaf(sq[d] * rq, s, a);
            }
        }
        for (int d = warp + 8 * kKeep; d < p.dim; d += 8) {
            const float s = fmaf(sk[d] * rk, u, fresh ? 0.f : g * S[(size_t)d * p.vdim]);
            S[(size_t)d * p.vdim] = s;
            a = fmaf(sq[d] * rq, s, a);
        }
    }
    __syncthreads();
    part[warp][lane] = a;
    __syncthreads();
    if (warp == 0 && live) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w][lane];
        p.o[(size_t)m * p.ldo + h * p.vdim + v] = o;
    }
}

// ---- token blocks ------------------------------------------------------------------------------------------------------

// columns c .. c + 3 of a row of n
template <bool VEC>
__device__ __forceinline__ void store4(float* row, int c, int n, const float* f) {
    if (VEC && c + 4 <= n) {
        *reinterpret_cast<float4*>(row + c) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (c + e < n) row[c + e] = f[e];
    }
}

// Convolution, activation and norms of the block's tokens, their gates: a warp per (head of q, k or v; four tokens), four channels per
// lane and pass.  TAPS taps (0: any number) stay in registers with the rows they are applied to.
constexpr int kWarpTokens = 4;

__device__ __forceinline__ float fast_siluf(float z) { return __fdividef(z, 1.f + expf(-z)); }

template <bool VEC, int TAPS>
__global__ void __launch_bounds__(256) lb_delta_tokens_kernel(const LbDelta p, const LbDeltaBlock b, int T, int pos0) {
    constexpr int N = kWarpTokens;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, slots = 2 * p.kv_heads + p.heads, nch = lb_delta_channels(p);
    const int t0 = (blockIdx.x * 8 + warp) * N, slot = blockIdx.y;
    if (t0 >= T) return;
    if (slot == slots) {  // the last row of CTAs makes the gates
        for (int i = lane; i < N * p.heads; i += 32) {
            const int t = t0 + i / p.heads, h = i % p.heads;
            if (t >= T) break;
            const float* row = p.proj + (size_t)t * p.ldp;
            b.beta[(size_t)t * p.heads + h] = write_strength(p, row, h);
            b.logg[(size_t)t * p.heads + h] = log_gate(p, row, h);
        }
        return;
    }
    const bool value = slot >= 2 * p.kv_heads;
    const int n = value ? p.vdim : p.dim, c0 = value ? 2 * p.kv_heads * p.dim + (slot - 2 * p.kv_heads) * p.vdim : slot * p.dim;
    float* out = b.qkv + (size_t)t0 * nch + c0;
    auto read = [&](int t, int c, float* y) {  // projections of the block's token t, of an earlier one (in the ring), or before the start
        if (pos0 + t < 0 || t >= T)
            y[0] = y[1] = y[2] = y[3] = 0.f;
        else
            lb_load_cols<4>(t >= 0 ? p.proj + (size_t)t * p.ldp + c0 : p.ring + (size_t)((pos0 + t) % p.taps) * nch + c0, c, n, VEC, y);
    };
    float ss[N] = {};
    for (int c = lane * 4; c < n; c += 128) {
        float a[N][4] = {};
        if (TAPS > 0) {
            constexpr int K = TAPS > 0 ? TAPS : 1;
            float w[K][4], y[N + K - 1][4];
#pragma unroll
            for (int j = 0; j < K; ++j) lb_load_cols<4>(p.conv_w + (size_t)j * nch + c0, c, n, VEC, w[j]);
#pragma unroll
            for (int j = 0; j < N + K - 1; ++j) read(t0 - (K - 1) + j, c, y[j]);
#pragma unroll
            for (int i = 0; i < N; ++i)
#pragma unroll
                for (int j = 0; j < K; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) a[i][e] = fmaf(w[j][e], y[i + j][e], a[i][e]);
        } else {
            for (int j = 0; j < p.taps; ++j) {  // tap j looks back taps - 1 - j positions
                float w[4], y[4];
                lb_load_cols<4>(p.conv_w + (size_t)j * nch + c0, c, n, VEC, w);
#pragma unroll
                for (int i = 0; i < N; ++i) {
                    read(t0 + i - (p.taps - 1) + j, c, y);
#pragma unroll
                    for (int e = 0; e < 4; ++e) a[i][e] = fmaf(w[e], y[e], a[i][e]);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < N; ++i) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                a[i][e] = fast_siluf(a[i][e]);  // (zero behind the last channel)
                ss[i] = fmaf(a[i][e], a[i][e], ss[i]);
            }
            if (t0 + i < T) store4<VEC>(out + (size_t)i * nch, c, n, a[i]);
        }
    }
    if (value) return;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const float r = __fdiv_rn(slot < p.kv_heads ? p.qscale : 1.f, sqrtf(lb_warp_sumf(ss[i]) + kUnitEps));
        if (t0 + i >= T) break;
        for (int c = lane * 4; c < n; c += 128) {  // (a thread reads back what it wrote)
            float a[4];
            lb_load_cols<4>(out + (size_t)i * nch, c, n, VEC, a);
#pragma unroll
            for (int e = 0; e < 4; ++e) a[e] *= r;
            store4<VEC>(out + (size_t)i * nch, c, n, a);
        }
    }
}

// the last taps - 1 projections of the block into the ring (after every token has been through its convolution)
__global__ void __launch_bounds__(256) lb_delta_commit_kernel(const LbDelta p, int T, int pos0) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = T - 1 - (int)blockIdx.y, c = blockIdx.x * 256 + threadIdx.x, nch = lb_delta_channels(p);
    if (t < 0 || c >= nch) return;
    p.ring[(size_t)((pos0 + t) % p.taps) * nch + c] = p.proj[(size_t)t * p.ldp + c];
}

__host__ __device__ inline int lead(int dim) { return lb_round_up(dim, 4) + 4; }

// acc[i][e] += sum over s of m[ty + 16 i][s] x[s][col + e] for a lower triangular m (its upper blocks are never read)
template <int NI>
__device__ __forceinline__ void tri_mul(const float* m, int ldm, const float* x, int ldx, int ty, int col, float (*acc)[4]) {
#pragma unroll
    for (int sb = 0; sb < NI; ++sb)
#pragma unroll
        for (int s = sb * 16; s < sb * 16 + 16; s += 4) {
            float4 w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) w[e] = *reinterpret_cast<const float4*>(x + (s + e) * ldx + col);
#pragma unroll
            for (int i = sb; i < NI; ++i) {
                const float4 a = *reinterpret_cast<const float4*>(m + (ty + 16 * i) * ldm + s);
                const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[i][0] = fmaf(av[e], w[e].x, acc[i][0]);
                    acc[i][1] = fmaf(av[e], w[e].y, acc[i][1]);
                    acc[i][2] = fmaf(av[e], w[e].z, acc[i][2]);
                    acc[i][3] = fmaf(av[e], w[e].w, acc[i][3]);
                }
            }
        }
}

// (I + L)^-1 in place of the strictly lower triangular L [C][ld]: blocks of sixteen by substitution, a thread per column, then pairs of
// blocks of 16 and of 32: the lower left block of the inverse is -T22 L21 T11.  x: C/2 * C/2 floats
template <int C>
__device__ __forceinline__ void invert(float* l, int ld, float* x, int tid) {
    const int blk = tid >> 4, j = tid & 15;
    float c[16];
    if (blk < C / 16) {
        const float* b = l + (blk * 16) * ld + blk * 16;
#pragma unroll
        for (int t = 0; t < 16; ++t) {
            float a = t == j ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < t; ++s) a = fmaf(-b[t * ld + s], c[s], a);
            c[t] = a;
        }
    }
    __syncthreads();
    if (blk < C / 16)
#pragma unroll
        for (int t = 0; t < 16; ++t) l[(blk * 16 + t) * ld + blk * 16 + j] = c[t];
    __syncthreads();
#pragma unroll
    for (int n = 16; n < C; n *= 2) {
        for (int i = tid; i < C / (2 * n) * n * n; i += 256) {  // X = L21 T11
            const int q = i / (n * n), r = i / n % n, k = i % n;
            const float *l21 = l + (2 * q * n + n + r) * ld + 2 * q * n, *t11 = l + 2 * q * n * ld + 2 * q * n + k;
            float a = 0.f;
            for (int e = 0; e < n; ++e) a = fmaf(l21[e], t11[e * ld], a);  // (T11 is zero above its diagonal)
            x[i] = a;
        }
        __syncthreads();
        for (int i = tid; i < C / (2 * n) * n * n; i += 256) {
            const int q = i / (n * n), r = i / n % n, k = i % n;
            const float* t22 = l + (2 * q * n + n + r) * ld + 2 * q * n + n;
            float a = 0.f;
            for (int e = 0; e < n; ++e) a = fmaf(-t22[e], x[q * n * n + e * n + k], a);
            l[(2 * q * n + n + r) * ld + 2 * q * n + k] = a;
        }
        __syncthreads();
    }
}

constexpr int kValueCols = 64;                 // value columns of a pass
constexpr int kValueLd = kValueCols + 4;

// CTA = (chunk, head): L and A, the substitution, and the operands of the products over chunks
template <int C>
__global__ void __launch_bounds__(256, 2) lb_delta_prep_kernel(const LbDelta p, const LbDeltaBlock b, int T, bool vec) {
    extern __shared__ __align__(16) float sm[];
    __shared__ double s_log[C];
    __shared__ float s_beta[C], s_g[C], s_end[C];
    constexpr int NI = C / 16, LC = C + 4;
    const int ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, ty = tid >> 4, tx = tid & 15, dim = p.dim, LD = lead(dim), D4 = lb_round_up(dim, 4) / 4;
    const int hk = h / (p.heads / p.kv_heads), nch = lb_delta_channels(p), QK = p.kv_heads * dim, t0 = ch * C, n = min(C, T - t0);
    float *sk = sm, *sl = sk + C * LD, *sa = sl + C * LC, *sq = sa + C * LC;  // sq: also value columns [C][kValueLd], and scratch of the inversion
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    for (int i = tid; i < C * D4; i += 256) {
        const int t = i / D4, d = (i - t * D4) * 4;
        float q[4] = {0.f, 0.f, 0.f, 0.f}, k[4] = {0.f, 0.f, 0.f, 0.f};
        if (t < n) {
            const float* row = b.qkv + (size_t)(t0 + t) * nch + hk * dim;
            lb_load_cols<4>(row, d, dim, vec, q);
            lb_load_cols<4>(row + QK, d, dim, vec, k);
        }
        *reinterpret_cast<float4*>(sq + t * LD + d) = make_float4(q[0], q[1], q[2], q[3]);
        *reinterpret_cast<float4*>(sk + t * LD + d) = make_float4(k[0], k[1], k[2], k[3]);
    }
    if (tid < C) {
        s_beta[tid] = tid < n ? b.beta[(size_t)(t0 + tid) * p.heads + h] : 0.f;
        s_log[tid] = tid < n ? (double)b.logg[(size_t)(t0 + tid) * p.heads + h] : 0.0;
    }
    __syncthreads();
    if (tid < 32) {  // running sums: C / 32 tokens per lane, then over the lanes
        constexpr int PER = C < 32 ? 1 : C / 32;
        double v[PER], run = 0.0;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int t = tid * PER + i;
            run += t < C ? s_log[t] : 0.0;
            v[i] = run;
        }
        double before = run;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double up = __shfl_up_sync(0xffffffffu, before, o);
            if (tid >= o) before += up;
        }
        before -= run;
#pragma unroll
        for (int i = 0; i < PER; ++i)
            if (tid * PER + i < C) s_log[tid * PER + i] = before + v[i];
    }
    __syncthreads();
    if (tid < C) {
        s_g[tid] = expf((float)s_log[tid]);
        s_end[tid] = expf((float)(s_log[C - 1] - s_log[tid]));
    }
    {
        float qk[NI][NI] = {}, kk[NI][NI] = {};
#pragma unroll 2
        for (int d = 0; d < dim; d += 4) {  // (columns dim .. are zero)
            float4 q[NI], a[NI], k[NI];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                q[i] = *reinterpret_cast<const float4*>(sq + (ty + 16 * i) * LD + d);
                a[i] = *reinterpret_cast<const float4*>(sk + (ty + 16 * i) * LD + d);
                k[i] = *reinterpret_cast<const float4*>(sk + (tx + 16 * i) * LD + d);
            }
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j <= i; ++j) {
                    qk[i][j] = fmaf(q[i].x, k[j].x, fmaf(q[i].y, k[j].y, fmaf(q[i].z, k[j].z, fmaf(q[i].w, k[j].w, qk[i][j]))));
                    kk[i][j] = fmaf(a[i].x, k[j].x, fmaf(a[i].y, k[j].y, fmaf(a[i].z, k[j].z, fmaf(a[i].w, k[j].w, kk[i][j]))));
                }
        }
        float* A = b.c.weights + ((size_t)ch * p.heads + h) * C * C;
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int j = 0; j < NI; ++j) {
                const int t = ty + 16 * i, s = tx + 16 * j;
                float l = 0.f, w = 0.f;
                if (j <= i && s <= t && t < n) {
                    const float r = expf((float)(s_log[t] - s_log[s]));
                    w = r * qk[i][j];
                    if (s < t) l = s_beta[t] * r * kk[i][j];
                }
                sl[t * LC + s] = l;
                sa[t * LC + s] = -w;
                A[t * C + s] = w;
            }
    }
    __syncthreads();
    if (tid == 0) b.c.decay[(size_t)ch * p.heads + h] = s_g[C - 1];
    // keys decayed to the chunk's end; the keys in shared memory become beta G k, and queries go out of the way of the inversion
    for (int i = tid; i < C * D4; i += 256) {
        const int t = i / D4, d = (i - t * D4) * 4;
        const float4 k = *reinterpret_cast<const float4*>(sk + t * LD + d);
        const float e = s_end[t], g = s_beta[t] * s_g[t], f[4] = {k.x * e, k.y * e, k.z * e, k.w * e};
        if (t < n) {
            float* out = b.c.kd + ((size_t)(t0 + t) * p.heads + h) * dim;
            if (vec)
                store4<true>(out, d, dim, f);
            else
                store4<false>(out, d, dim, f);
        }
        *reinterpret_cast<float4*>(sk + t * LD + d) = make_float4(k.x * g, k.y * g, k.z * g, k.w * g);
    }
    invert<C>(sl, LC, sq + C * (LD > kValueLd ? LD : kValueLd), tid);
    for (int d = tx * 4, d0 = 0; d0 < dim; d += 64, d0 += 64) {  // Wk, in place of the keys, and the queries against the state
        float acc[NI][4] = {};
        if (d < dim) tri_mul<NI>(sl, LC, sk, LD, ty, d, acc);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            if (d >= dim) continue;
            *reinterpret_cast<float4*>(sk + t * LD + d) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
            if (t >= n) continue;
            float* out = b.wk + ((size_t)(t0 + t) * p.heads + h) * dim;
            if (vec)
                store4<true>(out, d, dim, acc[i]);
            else
                store4<false>(out, d, dim, acc[i]);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const float4 q = *reinterpret_cast<const float4*>(sq + (ty + 16 * i) * LD + (d < dim ? d : 0));
            const float g = s_g[ty + 16 * i];
            acc[i][0] = g * q.x;
            acc[i][1] = g * q.y;
            acc[i][2] = g * q.z;
            acc[i][3] = g * q.w;
        }
        if (d >= dim) continue;
        tri_mul<NI>(sa, LC, sk, LD, ty, d, acc);  // (sa holds -A)
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            if (t >= n) continue;
            float* out = b.c.qd + ((size_t)(t0 + t) * p.heads + h) * dim;
            if (vec)
                store4<true>(out, d, dim, acc[i]);
            else
                store4<false>(out, d, dim, acc[i]);
        }
    }
    const float* v = b.qkv + (size_t)t0 * nch + 2 * QK + h * p.vdim;
    float f[NI][4];
    auto read = [&](int v0) {
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            if (t < n)
                lb_load_cols<4>(v + (size_t)t * nch, v0 + tx * 4, p.vdim, vec, f[i]);
            else
                f[i][0] = f[i][1] = f[i][2] = f[i][3] = 0.f;
        }
    };
    read(0);
    for (int v0 = 0; v0 < p.vdim; v0 += kValueCols) {
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            const float x = s_beta[t];
            *reinterpret_cast<float4*>(sq + t * kValueLd + tx * 4) = make_float4(f[i][0] * x, f[i][1] * x, f[i][2] * x, f[i][3] * x);
        }
        __syncthreads();
        if (v0 + kValueCols < p.vdim) read(v0 + kValueCols);
        float acc[NI][4] = {};
        tri_mul<NI>(sl, LC, sq, kValueLd, ty, tx * 4, acc);
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            if (t >= n) continue;
            float* out = b.wv + ((size_t)(t0 + t) * p.heads + h) * p.vdim;
            if (vec)
                store4<true>(out, v0 + tx * 4, p.vdim, acc[i]);
            else
                store4<false>(out, v0 + tx * 4, p.vdim, acc[i]);
        }
    }
}

// ---- the states in front of the chunks, one after the other: CTA = (a few value columns, head) ---------------------------
//
// S <- G S + N - M S with M = Kd^T Wk (dim x dim) and N = Kd^T Wv.  Panels of up to 128 rows of M and the columns of N travel while
// the panel before is worked on; the old and the new state are in shared memory.  A lane has two rows of the panel and all of the CTA's
// columns, so that a row of the old state is one broadcast for a whole warp; two warps have the panel's rows, kScanSplit such pairs split
// the sum over the old state's rows.
constexpr size_t kScanSmem = 224 * 1024;
constexpr int kScanRows = 2, kScanSplit = 4, kScanWarps = 2 * kScanSplit;

__device__ __forceinline__ void copy_async(float* dst, const float* src, bool wide) {
    if (wide)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(lb_smem_u32(dst)), "l"(src) : "memory");
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(lb_smem_u32(dst)), "l"(src) : "memory");
}

// floats of a panel's buffer: the panel, later the warps' sums
__host__ __device__ inline int scan_buffer(int dim, int panel, int cols) { return panel * (lead(dim) > kScanSplit * cols ? lead(dim) : kScanSplit * cols); }
size_t scan_smem(int dim, int panel, int cols) { return ((size_t)2 * scan_buffer(dim, panel, cols) + (size_t)4 * lb_round_up(dim, 4) * cols) * sizeof(float); }
struct ScanShape {
    int panel, cols;
};
// as few columns as keep every SM busy once, in panels as high as fit; panel 0: does not fit
ScanShape scan_shape(int dim, int vdim, int heads, int sms) {
    const int per_head = sms / heads > 1 ? sms / heads : 1;
    int cols = lb_round_up(lb_ceil_div(vdim, per_head), 4);
    if (cols > 32) cols = 32;
    int want = 128;
    while (want > 32 && want / 2 >= dim) want /= 2;
    for (; cols >= 4; cols -= 4) {
        int panel = want;
        while (panel > 4 && scan_smem(dim, panel, cols) > kScanSmem) panel /= 2;
        if (scan_smem(dim, panel, cols) > kScanSmem) continue;
        if (panel >= 32 || cols == 4) return {panel, cols};
    }
    return {0, 0};
}

template <int COLS>
__global__ void __launch_bounds__(kScanWarps * 32, 1) lb_delta_scan_kernel(const LbDeltaBlock b, int chunks, int panel, int fresh, bool wide_m, bool wide_n) {
    extern __shared__ __align__(16) float sm[];
    constexpr int NT = kScanWarps * 32;
    const LbChunks& c = b.c;
    const int dim = c.dim, vdim = c.vdim, LD = lead(dim), DP = lb_round_up(dim, 4), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.y, v0 = blockIdx.x * COLS;
    const int buffer = scan_buffer(dim, panel, COLS);
    float *sM = sm, *sN = sM + 2 * buffer, *sS = sN + 2 * DP * COLS;
    const int panels = lb_ceil_div(dim, panel), steps = chunks * panels, live = min(COLS, vdim - v0);
    for (int i = tid; i < 2 * buffer + 4 * DP * COLS; i += NT) sm[i] = 0.f;
    __syncthreads();
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    float* S0 = c.state + (size_t)h * dim * vdim + v0;
    if (!fresh)
        for (int i = tid; i < dim * COLS; i += NT) {
            const int d = i / COLS, v = i % COLS;
            if (v < live) sS[i] = S0[(size_t)d * vdim + v];
        }
    const int qm = wide_m ? 4 : 1, qn = wide_n ? 4 : 1;
    auto fetch = [&](int step) {
        const int cc = step / panels, d0 = (step - cc * panels) * panel, rows = min(panel, dim - d0);
        const float* M = b.mix + (((size_t)cc * c.heads + h) * dim + d0) * dim;
        float* dst = sM + (step & 1) * buffer;
        if (wide_m && dim == 128) {
            dst += warp * LD + lane * 4;
            M += warp * 128 + lane * 4;
#pragma unroll 4
            for (int r = warp; r < rows; r += kScanWarps, dst += kScanWarps * LD, M += kScanWarps * 128) copy_async(dst, M, true);
        } else {
            for (int r = warp; r < rows; r += kScanWarps)
                for (int e = lane * qm; e < dim; e += 32 * qm) copy_async(dst + r * LD + e, M + (size_t)r * dim + e, wide_m);
        }
        if (d0 == 0) {
            const float* N = c.states + ((size_t)cc * c.heads + h) * dim * vdim + v0;
            float* to = sN + (cc & 1) * DP * COLS;
            for (int i = tid; i < dim * (COLS / qn); i += NT) {
                const int d = i / (COLS / qn), v = (i - d * (COLS / qn)) * qn;
                if (v < live) copy_async(to + d * COLS + v, N + (size_t)d * vdim + v, wide_n);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const int part = warp >> 1, row0 = (warp & 1) * 32 * kScanRows + lane, e0 = DP / 4 * part / kScanSplit * 4, e1 = DP / 4 * (part + 1) / kScanSplit * 4;
    fetch(0);
    for (int step = 0; step < steps; ++step) {
        const int cc = step / panels, d0 = (step - cc * panels) * panel, rows = min(panel, dim - d0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the panel is here, and everyone is done with the other buffer
        if (step + 1 < steps) fetch(step + 1);
        const float g = c.decay[(size_t)cc * c.heads + h];
        const float *S = sS + (cc & 1) * DP * COLS, *N = sN + (cc & 1) * DP * COLS;
        float* M = sM + (step & 1) * buffer;
        uint64_t acc[kScanRows][COLS / 2] = {};  // pairs of columns
#pragma unroll 2
        for (int e = e0; e < e1; e += 4) {
            float m[kScanRows][4];
#pragma unroll
            for (int i = 0; i < kScanRows; ++i) {
                const float4 x = row0 + 32 * i < rows ? *reinterpret_cast<const float4*>(M + (row0 + 32 * i) * LD + e) : make_float4(0.f, 0.f, 0.f, 0.f);
                m[i][0] = x.x;
                m[i][1] = x.y;
                m[i][2] = x.z;
                m[i][3] = x.w;
            }
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                uint64_t mm[kScanRows];
#pragma unroll
                for (int i = 0; i < kScanRows; ++i) mm[i] = lb_pack2(m[i][k], m[i][k]);
#pragma unroll
                for (int v = 0; v < COLS; v += 4) {
                    const ulonglong2 s = *reinterpret_cast<const ulonglong2*>(S + (e + k) * COLS + v);
#pragma unroll
                    for (int i = 0; i < kScanRows; ++i) {
                        acc[i][v / 2] = lb_fma2(mm[i], s.x, acc[i][v / 2]);
                        acc[i][v / 2 + 1] = lb_fma2(mm[i], s.y, acc[i][v / 2 + 1]);
                    }
                }
            }
        }
        __syncthreads();  // the panel has been read: its buffer takes the warps' sums [part][column / 4][row][4]
#pragma unroll
        for (int i = 0; i < kScanRows; ++i)
            if (row0 + 32 * i < rows)
#pragma unroll
                for (int v = 0; v < COLS; v += 4)
                    *reinterpret_cast<ulonglong2*>(M + ((part * (COLS / 4) + v / 4) * panel + row0 + 32 * i) * 4) = make_ulonglong2(acc[i][v / 2], acc[i][v / 2 + 1]);
        __syncthreads();
        float* next = sS + ((cc + 1) & 1) * DP * COLS;
        float* out = c.states + ((size_t)cc * c.heads + h) * dim * vdim + v0;
        for (int i = tid; i < rows * (COLS / 4); i += NT) {
            const int q = i / rows, r = i - q * rows, v = q * 4, d = d0 + r;
            float4 x = *reinterpret_cast<const float4*>(M + (q * panel + r) * 4);
#pragma unroll
            for (int w = 1; w < kScanSplit; ++w) {
                const float4 y = *reinterpret_cast<const float4*>(M + ((w * (COLS / 4) + q) * panel + r) * 4);
                x = make_float4(x.x + y.x, x.y + y.y, x.z + y.z, x.w + y.w);
            }
            const float4 old = *reinterpret_cast<const float4*>(S + d * COLS + v), add = *reinterpret_cast<const float4*>(N + d * COLS + v);
            *reinterpret_cast<float4*>(next + d * COLS + v) =
                make_float4(fmaf(g, old.x, add.x - x.x), fmaf(g, old.y, add.y - x.y), fmaf(g, old.z, add.z - x.z), fmaf(g, old.w, add.w - x.w));
            const float o[4] = {old.x, old.y, old.z, old.w};
            if (wide_n)
                store4<true>(out + (size_t)d * vdim, v, live, o);
            else
                store4<false>(out + (size_t)d * vdim, v, live, o);
        }
    }
    __syncthreads();
    const float* last = sS + (chunks & 1) * DP * COLS;
    for (int i = tid; i < dim * COLS; i += NT) {
        const int d = i / COLS, x = i % COLS;
        if (x < live) S0[(size_t)d * vdim + x] = last[i];
    }
}

template <int COLS>
int launch_scan(loom_b200_ctx* ctx, const LbDeltaBlock& b, int chunks, int panel, bool fresh) {
    LB_BIG_SMEM(ctx, lb_delta_scan_kernel<COLS>, kScanSmem);
    LB_LAUNCH(ctx, lb_delta_scan_kernel<COLS>, dim3(lb_ceil_div(b.c.vdim, COLS), b.c.heads), dim3(kScanWarps * 32), scan_smem(b.c.dim, panel, COLS), b, chunks, panel, fresh ? 1 : 0,
              b.c.dim % 4 == 0, b.c.vdim % 4 == 0);
    return 0;
}
int run_scan(loom_b200_ctx* ctx, const LbDeltaBlock& b, int chunks, bool fresh) {
    const ScanShape s = scan_shape(b.c.dim, b.c.vdim, b.c.heads, ctx->sm_count);
    switch (s.cols) {
        case 4: return launch_scan<4>(ctx, b, chunks, s.panel, fresh);
        case 8: return launch_scan<8>(ctx, b, chunks, s.panel, fresh);
        case 12: return launch_scan<12>(ctx, b, chunks, s.panel, fresh);
        case 16: return launch_scan<16>(ctx, b, chunks, s.panel, fresh);
        case 20: return launch_scan<20>(ctx, b, chunks, s.panel, fresh);
        case 24: return launch_scan<24>(ctx, b, chunks, s.panel, fresh);
        case 28: return launch_scan<28>(ctx, b, chunks, s.panel, fresh);
        case 32: return launch_scan<32>(ctx, b, chunks, s.panel, fresh);
    }
    return lb_fail(ctx, LOOM_B200_ERR_UNSUPPORTED, "delta rule: %d key channels", b.c.dim);
}

size_t prep_smem(int C, int dim) {
    const size_t q = lead(dim) > kValueLd ? lead(dim) : kValueLd;
    return ((size_t)C * lead(dim) + (size_t)C * q + (size_t)2 * C * (C + 4) + (size_t)C * C / 4) * sizeof(float);
}

template <int C>
int launch_prep(loom_b200_ctx* ctx, const LbDelta& p, const LbDeltaBlock& b, int T, bool vec) {
    LB_BIG_SMEM(ctx, lb_delta_prep_kernel<C>, 200 * 1024);
    LB_LAUNCH(ctx, lb_delta_prep_kernel<C>, dim3(lb_ceil_div(T, C), p.heads), dim3(256), prep_smem(C, p.dim), p, b, T, vec);
    return 0;
}

}  // namespace

int lb_delta_chunk(int dim) {
    if (!scan_shape(dim, 4, 1, 148).panel) return 0;
    for (int C = 64; C >= 16; C /= 2)
        if (prep_smem(C, dim) <= 200 * 1024) return C;
    return 0;
}

int lb_delta_step(loom_b200_ctx* ctx, const LbDelta& p, const int* pos, int lane0, int M) {
    const size_t smem = (size_t)2 * p.dim * sizeof(float);
    LB_REQUIRE(ctx, smem <= 40 * 1024 && p.taps >= 1 && p.taps <= kMaxTaps, "delta rule: %d key channels, %d taps", p.dim, p.taps);
    LB_LAUNCH(ctx, lb_delta_step_kernel, dim3(lb_ceil_div(p.vdim, 32), p.heads, M), dim3(256), smem, p, pos, lane0);
    return 0;
}

int lb_delta_block(loom_b200_ctx* ctx, const LbDelta& p, const LbDeltaBlock& bin, int T, int pos0) {
    LbDeltaBlock b = bin;
    b.c.C = lb_delta_chunk(p.dim);
    LB_REQUIRE(ctx, b.c.C > 0 && p.taps >= 1 && p.taps <= kMaxTaps, "delta rule: %d key channels, %d taps", p.dim, p.taps);
    b.c.heads = p.heads;
    b.c.dim = p.dim;
    b.c.vdim = p.vdim;
    b.c.v = b.wv;
    b.c.ldv = p.heads * p.vdim;
    b.c.state = p.state;
    b.c.o = p.o;
    b.c.ldo = p.ldo;
    const int chunks = lb_ceil_div(T, b.c.C);
    const bool vec = p.dim % 4 == 0 && p.vdim % 4 == 0 && lb_vec_rows(p.proj, p.ldp);
    const dim3 tokens(lb_ceil_div(T, 8 * kWarpTokens), 2 * p.kv_heads + p.heads + 1);
    if (vec && p.taps == 4)
        LB_LAUNCH(ctx, (lb_delta_tokens_kernel<true, 4>), tokens, dim3(256), 0, p, b, T, pos0);
    else if (vec)
        LB_LAUNCH(ctx, (lb_delta_tokens_kernel<true, 0>), tokens, dim3(256), 0, p, b, T, pos0);
    else
        LB_LAUNCH(ctx, (lb_delta_tokens_kernel<false, 0>), tokens, dim3(256), 0, p, b, T, pos0);
    if (p.taps > 1) LB_LAUNCH(ctx, lb_delta_commit_kernel, dim3(lb_ceil_div(lb_delta_channels(p), 256), p.taps - 1), dim3(256), 0, p, T, pos0);
    int rc = b.c.C == 64 ? launch_prep<64>(ctx, p, b, T, vec) : b.c.C == 32 ? launch_prep<32>(ctx, p, b, T, vec) : launch_prep<16>(ctx, p, b, T, vec);
    if (rc) return rc;
    if ((rc = lb_chunk_states(ctx, b.c, T))) return rc;
    LbChunks m = b.c;  // what a chunk takes out of the state
    m.vdim = p.dim;
    m.v = b.wk;
    m.ldv = p.heads * p.dim;
    m.states = b.mix;
    if ((rc = lb_chunk_states(ctx, m, T))) return rc;
    if ((rc = run_scan(ctx, b, chunks, pos0 == 0))) return rc;
    return lb_chunk_out(ctx, b.c, T);
}
