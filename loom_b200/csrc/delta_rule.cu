// delta_rule.cu -- gated delta rule with one decay per head behind short convolutions: the one-token step and the token block.
//
//   S' = g_t S_(t-1),  u_t = beta_t (v_t - S'^T k_t),  S_t = S' + k_t u_t^T,  o_t = S_t^T q_t
//
// A block of tokens is cut into chunks of C.  With G_t the product of the decays inside a chunk and S the state in front of it,
//   u_t + sum_(s < t) L_ts u_s = beta_t v_t - beta_t G_t S^T k_t,   L_ts = beta_t (G_t / G_s) k_t.k_s
// so forward substitution with L on the columns of (beta v | beta G k) gives u = Wv - Wk S without knowing S, and
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

constexpr int kRows = 8;  // tokens of a CTA

// convolution, activation and norms of the block's tokens, their gates: a warp per (head of q, k or v; token)
__global__ void __launch_bounds__(256) lb_delta_tokens_kernel(const LbDelta p, const LbDeltaBlock b, int T, int pos0) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t0 = blockIdx.x * kRows, rows = min(kRows, T - t0);
    const int nch = lb_delta_channels(p), slots = 2 * p.kv_heads + p.heads, back = p.taps - 1;
    for (int i = warp; i < slots * kRows; i += 8) {
        const int slot = i / kRows, t = t0 + i % kRows;
        if (t >= T) continue;
        const bool value = slot >= 2 * p.kv_heads;
        const int n = value ? p.vdim : p.dim, c0 = value ? 2 * p.kv_heads * p.dim + (slot - 2 * p.kv_heads) * p.vdim : slot * p.dim;
        float* out = b.qkv + (size_t)t * nch + c0;
        const float *x = p.proj + c0, *w = p.conv_w + c0;
        float ss = 0.f;
        for (int c = lane; c < n; c += 32) {
            float a = 0.f;
#pragma unroll 4
            for (int j = 0; j <= back; ++j) {
                const int ts = t - back + j;
                if (pos0 + ts < 0) continue;
                const float y = ts >= 0 ? x[(size_t)ts * p.ldp + c] : p.ring[(size_t)((pos0 + ts) % p.taps) * nch + c0 + c];
                a = fmaf(w[(size_t)j * nch + c], y, a);
            }
            a = lb_siluf(a);
            out[c] = a;
            ss = fmaf(a, a, ss);
        }
        if (value) continue;
        ss = lb_warp_sumf(ss);
        const float r = __fdiv_rn(slot < p.kv_heads ? p.qscale : 1.f, sqrtf(ss + kUnitEps));
        for (int c = lane; c < n; c += 32) out[c] *= r;  // (a thread reads back what it wrote)
    }
    for (int i = threadIdx.x; i < rows * p.heads; i += 256) {
        const int t = t0 + i / p.heads, h = i % p.heads;
        const float* row = p.proj + (size_t)t * p.ldp;
        b.beta[(size_t)t * p.heads + h] = write_strength(p, row, h);
        b.logg[(size_t)t * p.heads + h] = log_gate(p, row, h);
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

// CTA = (chunk, head): L and A, the substitution, and the operands of the products over chunks
template <int C>
__global__ void __launch_bounds__(256, 2) lb_delta_prep_kernel(const LbDelta p, const LbDeltaBlock b, int T) {
    extern __shared__ __align__(16) float sm[];
    __shared__ double s_log[C];
    __shared__ float s_beta[C], s_g[C];
    constexpr int NI = C / 16, LC = C + 4;
    const int ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, dim = p.dim, LD = lead(dim);
    const int hk = h / (p.heads / p.kv_heads), nch = lb_delta_channels(p), QK = p.kv_heads * dim, t0 = ch * C, n = min(C, T - t0);
    float *sq = sm, *sk = sq + C * LD, *sl = sk + C * LD, *sa = sl + C * LC;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    for (int i = tid; i < C * LD; i += 256) {
        const int t = i / LD, d = i - t * LD;
        const bool ok = t < n && d < dim;
        const float* row = b.qkv + (size_t)(t0 + t) * nch + hk * dim + d;
        sq[i] = ok ? row[0] : 0.f;
        sk[i] = ok ? row[QK] : 0.f;
    }
    if (tid < C) {
        s_beta[tid] = tid < n ? b.beta[(size_t)(t0 + tid) * p.heads + h] : 0.f;
        s_log[tid] = tid < n ? (double)b.logg[(size_t)(t0 + tid) * p.heads + h] : 0.0;
    }
    __syncthreads();
    if (tid == 0)
        for (int t = 1; t < C; ++t) s_log[t] += s_log[t - 1];
    __syncthreads();
    if (tid < C) s_g[tid] = expf((float)s_log[tid]);
    {
        const int ty = tid >> 4, tx = tid & 15;
        float qk[NI][NI] = {}, kk[NI][NI] = {};
        for (int d = 0; d < dim; d += 4) {  // (columns dim .. LD are zero)
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
                sa[t * LC + s] = w;
                A[t * C + s] = w;
            }
    }
    __syncthreads();
    if (tid == 0) b.c.decay[(size_t)ch * p.heads + h] = s_g[C - 1];
    for (int i = tid; i < n * dim; i += 256) {
        const int t = i / dim, d = i - t * dim;
        b.c.kd[((size_t)(t0 + t) * p.heads + h) * dim + d] = sk[t * LD + d] * expf((float)(s_log[C - 1] - s_log[t]));
    }
    __syncthreads();
    // a thread per column of (beta v | beta G k); the solved key columns replace the keys
    for (int col = tid; col < p.vdim + dim; col += 256) {
        const bool value = col < p.vdim;
        const int d = col - p.vdim;
        float w[C];
#pragma unroll
        for (int t = 0; t < C; ++t) {
            if (value)
                w[t] = t < n ? b.qkv[(size_t)(t0 + t) * nch + 2 * QK + h * p.vdim + col] * s_beta[t] : 0.f;
            else
                w[t] = sk[t * LD + d] * (s_beta[t] * s_g[t]);
        }
#pragma unroll
        for (int t = 1; t < C; ++t) {
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int s = 0; s < t; s += 4) {
                const float4 l = *reinterpret_cast<const float4*>(sl + t * LC + s);
                a0 = fmaf(l.x, w[s], a0);
                if (s + 1 < t) a1 = fmaf(l.y, w[s + 1], a1);
                if (s + 2 < t) a0 = fmaf(l.z, w[s + 2], a0);
                if (s + 3 < t) a1 = fmaf(l.w, w[s + 3], a1);
            }
            w[t] -= a0 + a1;
        }
#pragma unroll
        for (int t = 0; t < C; ++t) {
            if (value) {
                if (t < n) b.wv[(size_t)(t0 + t) * p.heads * p.vdim + h * p.vdim + col] = w[t];
            } else {
                sk[t * LD + d] = w[t];
                if (t < n) b.wk[((size_t)(t0 + t) * p.heads + h) * dim + d] = w[t];
            }
        }
    }
    __syncthreads();
    const int ty = tid >> 4, tx = tid & 15;
    for (int d = tx * 4; d < dim; d += 64) {
        float acc[NI][4];
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            const float4 q = *reinterpret_cast<const float4*>(sq + t * LD + d);
            acc[i][0] = s_g[t] * q.x;
            acc[i][1] = s_g[t] * q.y;
            acc[i][2] = s_g[t] * q.z;
            acc[i][3] = s_g[t] * q.w;
        }
#pragma unroll
        for (int sb = 0; sb < NI; ++sb)
#pragma unroll
            for (int s = sb * 16; s < sb * 16 + 16; s += 4) {
                float4 w[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) w[e] = *reinterpret_cast<const float4*>(sk + (s + e) * LD + d);
#pragma unroll
                for (int i = sb; i < NI; ++i) {
                    const float4 a = *reinterpret_cast<const float4*>(sa + (ty + 16 * i) * LC + s);
                    const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        acc[i][0] = fmaf(-av[e], w[e].x, acc[i][0]);
                        acc[i][1] = fmaf(-av[e], w[e].y, acc[i][1]);
                        acc[i][2] = fmaf(-av[e], w[e].z, acc[i][2]);
                        acc[i][3] = fmaf(-av[e], w[e].w, acc[i][3]);
                    }
                }
            }
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            const int t = ty + 16 * i;
            if (t >= n) continue;
            float* out = b.c.qd + ((size_t)(t0 + t) * p.heads + h) * dim + d;
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (d + e < dim) out[e] = acc[i][e];
        }
    }
}

// ---- the states in front of the chunks, one after the other: CTA = (16 value columns, head) ------------------------------
//
// S <- G S + N - M S with M = Kd^T Wk (dim x dim) and N = Kd^T Wv.  Panels of rows of M and the columns of N travel while the panel
// before is worked on; the old and the new state are in shared memory.
constexpr int kScanCols = 16;
constexpr size_t kScanSmem = 200 * 1024;

__device__ __forceinline__ void copy_async(float* dst, const float* src, bool wide) {
    if (wide)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(lb_smem_u32(dst)), "l"(src) : "memory");
    else
        asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(lb_smem_u32(dst)), "l"(src) : "memory");
}

size_t scan_smem(int dim, int panel) { return ((size_t)2 * panel * lead(dim) + (size_t)4 * lb_round_up(dim, 4) * kScanCols) * sizeof(float); }
int scan_panel(int dim) {
    int p = 128;
    while (p > 16 && p / 2 >= dim) p /= 2;
    while (p > 8 && scan_smem(dim, p) > kScanSmem) p /= 2;
    return scan_smem(dim, p) <= kScanSmem ? p : 0;
}

__global__ void __launch_bounds__(256) lb_delta_scan_kernel(const LbDeltaBlock b, int chunks, int panel, int fresh, bool wide_m, bool wide_n) {
    extern __shared__ __align__(16) float sm[];
    const LbChunks& c = b.c;
    const int dim = c.dim, vdim = c.vdim, LD = lead(dim), DP = lb_round_up(dim, 4), tid = threadIdx.x, h = blockIdx.y, v0 = blockIdx.x * kScanCols;
    float *sM = sm, *sN = sM + 2 * panel * LD, *sS = sN + 2 * DP * kScanCols;
    const int panels = lb_ceil_div(dim, panel), steps = chunks * panels, cols = min(kScanCols, vdim - v0);
    for (int i = tid; i < 2 * panel * LD + 4 * DP * kScanCols; i += 256) sm[i] = 0.f;
    __syncthreads();
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    float* S0 = c.state + (size_t)h * dim * vdim + v0;
    if (!fresh)
        for (int i = tid; i < dim * kScanCols; i += 256) {
            const int d = i / kScanCols, v = i % kScanCols;
            if (v < cols) sS[i] = S0[(size_t)d * vdim + v];
        }
    auto fetch = [&](int step) {
        const int cc = step / panels, d0 = (step - cc * panels) * panel, rows = min(panel, dim - d0);
        const float* M = b.mix + (((size_t)cc * c.heads + h) * dim + d0) * dim;
        float* dst = sM + (step & 1) * panel * LD;
        const int q = wide_m ? 4 : 1, per = dim / q;
        for (int i = tid; i < rows * per; i += 256) {
            const int r = i / per, e = (i - r * per) * q;
            copy_async(dst + r * LD + e, M + (size_t)r * dim + e, wide_m);
        }
        if (d0 == 0) {
            const float* N = c.states + ((size_t)cc * c.heads + h) * dim * vdim + v0;
            float* to = sN + (cc & 1) * DP * kScanCols;
            const int qn = wide_n ? 4 : 1, pn = cols / qn;
            for (int i = tid; i < dim * pn; i += 256) {
                const int d = i / pn, v = (i - d * pn) * qn;
                copy_async(to + d * kScanCols + v, N + (size_t)d * vdim + v, wide_n);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0);
    for (int step = 0; step < steps; ++step) {
        const int cc = step / panels, d0 = (step - cc * panels) * panel, rows = min(panel, dim - d0);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();  // the panel is here, and everyone is done with the other buffer
        if (step + 1 < steps) fetch(step + 1);
        const float *S = sS + (cc & 1) * DP * kScanCols, *N = sN + (cc & 1) * DP * kScanCols, *M = sM + (step & 1) * panel * LD;
        float* next = sS + ((cc + 1) & 1) * DP * kScanCols;
        const float g = c.decay[(size_t)cc * c.heads + h];
        float* out = c.states + ((size_t)cc * c.heads + h) * dim * vdim + v0;
        for (int i = tid; i < (panel / 2) * 4; i += 256) {
            const int r = (i >> 2) * 2, v = (i & 3) * 4;
            if (r >= rows) continue;
            const float *m0 = M + r * LD, *m1 = m0 + LD;  // (a row behind the last one holds finite leftovers and is not stored)
            float a0[4] = {}, a1[4] = {};
#pragma unroll 4
            for (int e = 0; e < DP; e += 4) {
                const float4 x = *reinterpret_cast<const float4*>(m0 + e), y = *reinterpret_cast<const float4*>(m1 + e);
                const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const float4 s = *reinterpret_cast<const float4*>(S + (e + k) * kScanCols + v);
                    a0[0] = fmaf(xv[k], s.x, a0[0]);
                    a0[1] = fmaf(xv[k], s.y, a0[1]);
                    a0[2] = fmaf(xv[k], s.z, a0[2]);
                    a0[3] = fmaf(xv[k], s.w, a0[3]);
                    a1[0] = fmaf(yv[k], s.x, a1[0]);
                    a1[1] = fmaf(yv[k], s.y, a1[1]);
                    a1[2] = fmaf(yv[k], s.z, a1[2]);
                    a1[3] = fmaf(yv[k], s.w, a1[3]);
                }
            }
#pragma unroll
            for (int rr = 0; rr < 2; ++rr) {
                const int d = d0 + r + rr;
                if (r + rr >= rows) continue;
                float old[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    old[k] = S[d * kScanCols + v + k];
                    next[d * kScanCols + v + k] = fmaf(g, old[k], N[d * kScanCols + v + k] - (rr ? a1[k] : a0[k]));
                }
                if (wide_n && v + 4 <= cols) {
                    *reinterpret_cast<float4*>(out + (size_t)d * vdim + v) = make_float4(old[0], old[1], old[2], old[3]);
                } else {
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        if (v + k < cols) out[(size_t)d * vdim + v + k] = old[k];
                }
            }
        }
    }
    __syncthreads();
    const float* last = sS + (chunks & 1) * DP * kScanCols;
    for (int i = tid; i < dim * kScanCols; i += 256) {
        const int d = i / kScanCols, v = i % kScanCols;
        if (v < cols) S0[(size_t)d * vdim + v] = last[i];
    }
}

size_t prep_smem(int C, int dim) { return ((size_t)2 * C * lead(dim) + (size_t)2 * C * (C + 4)) * sizeof(float); }

template <int C>
int launch_prep(loom_b200_ctx* ctx, const LbDelta& p, const LbDeltaBlock& b, int T) {
    LB_BIG_SMEM(ctx, lb_delta_prep_kernel<C>, 200 * 1024);
    LB_LAUNCH(ctx, lb_delta_prep_kernel<C>, dim3(lb_ceil_div(T, C), p.heads), dim3(256), prep_smem(C, p.dim), p, b, T);
    return 0;
}

}  // namespace

int lb_delta_chunk(int dim) {
    if (!scan_panel(dim)) return 0;
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
    LB_LAUNCH(ctx, lb_delta_tokens_kernel, dim3(lb_ceil_div(T, kRows)), dim3(256), 0, p, b, T, pos0);
    if (p.taps > 1) LB_LAUNCH(ctx, lb_delta_commit_kernel, dim3(lb_ceil_div(lb_delta_channels(p), 256), p.taps - 1), dim3(256), 0, p, T, pos0);
    int rc = b.c.C == 64 ? launch_prep<64>(ctx, p, b, T) : b.c.C == 32 ? launch_prep<32>(ctx, p, b, T) : launch_prep<16>(ctx, p, b, T);
    if (rc) return rc;
    if ((rc = lb_chunk_states(ctx, b.c, T))) return rc;
    LbChunks m = b.c;  // what a chunk takes out of the state
    m.vdim = p.dim;
    m.v = b.wk;
    m.ldv = p.heads * p.dim;
    m.states = b.mix;
    if ((rc = lb_chunk_states(ctx, m, T))) return rc;
    const int panel = scan_panel(p.dim);
    LB_BIG_SMEM(ctx, lb_delta_scan_kernel, kScanSmem);
    LB_LAUNCH(ctx, lb_delta_scan_kernel, dim3(lb_ceil_div(p.vdim, kScanCols), p.heads), dim3(256), scan_smem(p.dim, panel), b, chunks, panel, pos0 == 0 ? 1 : 0,
              p.dim % 4 == 0, p.vdim % 4 == 0);
    return lb_chunk_out(ctx, b.c, T);
}
