// gated_linear.cu -- gated linear attention with a decay per key channel: the one-token step and the token block.
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t,  a_t = sigmoid(z_t)^(1/tau)
//
// A block of tokens is cut into chunks of C.  With B_t the running sum of log a inside a chunk and S the state in front of it,
//   o_t   = (q_t e^(B_t))^T S + sum_(s <= t) A_ts v_s,   A_ts = sum_d q_td k_sd e^(B_td - B_sd)
//   S_end = diag(e^(B_end)) S + sum_s (k_s e^(B_end - B_s)) v_s^T
// so that everything but a short scan over the chunks is a product of matrices.  No exponent is ever positive: pairs of tokens
// in different sub-blocks of sixteen split their exponent at the border between them, pairs inside one take it directly.
// All of it is 32-bit floats.
#include "mixers.cuh"

namespace {

__device__ __forceinline__ float log_decay(const LbGla& p, const float* low, int ch) {
    const int hd = p.heads * p.dim;
    float z = 0.f;
    for (int r = 0; r < p.rank; ++r) z = fmaf(p.a2t[(size_t)r * hd + ch], low[r], z);
    return lb_log_sigmoidf(z + p.a2b[ch]) * p.inv_tau;
}

// one new token per sequence: CTA = (32 value columns, head, sequence); warps split the key channels
__global__ void __launch_bounds__(256) lb_gla_step_kernel(const LbGla p, const int* pos, int lane0) {
    extern __shared__ float sm[];
    __shared__ float part[8][32];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.y, m = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int HD = p.heads * p.dim, HV = p.heads * p.vdim;
    float *sq = sm, *sk = sm + p.dim, *sa = sk + p.dim, *low = sa + p.dim;
    const float* row = p.proj + (size_t)m * p.ldp;
    const int v = blockIdx.x * 32 + lane;
    const bool live = v < p.vdim, fresh = pos[m] == 0;
    float* S = p.state + (((size_t)(lane0 + m) * p.heads + h) * p.dim) * p.vdim + v;
    const float vv = live ? row[2 * HD + h * p.vdim + v] : 0.f;
    float first[8];  // the first state rows of this warp are on their way while the decays are computed
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = warp + 8 * i;
        first[i] = live && !fresh && d < p.dim ? S[(size_t)d * p.vdim] : 0.f;
    }
    for (int r = threadIdx.x; r < p.rank; r += blockDim.x) low[r] = row[2 * HD + 2 * HV + r];
    for (int d = threadIdx.x; d < p.dim; d += blockDim.x) {
        sq[d] = row[h * p.dim + d] * p.qscale;
        sk[d] = row[HD + h * p.dim + d];
    }
    __syncthreads();
    for (int d = threadIdx.x; d < p.dim; d += blockDim.x) sa[d] = expf(log_decay(p, low, h * p.dim + d));
    __syncthreads();
    float acc = 0.f;
    auto row_step = [&](int d, float old) {
        const float s = fmaf(sa[d], old, sk[d] * vv);
        S[(size_t)d * p.vdim] = s;
        acc = fmaf(sq[d], s, acc);
    };
    if (live) {
#pragma unroll
        for (int i = 0; i < 8; ++i)
            if (warp + 8 * i < p.dim) row_step(warp + 8 * i, first[i]);
#pragma unroll 8
        for (int d = warp + 64; d < p.dim; d += 8) row_step(d, fresh ? 0.f : S[(size_t)d * p.vdim]);
    }
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && live) {
        float o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += part[w][lane];
        p.o[(size_t)m * p.ldo + h * p.vdim + v] = o;
    }
}

constexpr int kSub = 16;

// CTA = (chunk, head): decays, the scaled queries and keys and the chunk's token-by-token weights
__global__ void __launch_bounds__(256) lb_gla_prep_kernel(const LbGla p, const LbGlaBlock b, int T) {
    extern __shared__ __align__(16) float sm[];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int C = b.C, ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, dim = p.dim, LD = lb_round_up(dim, 4) + 4;
    const int HD = p.heads * dim, HV = p.heads * p.vdim, t0 = ch * C, n = min(C, T - t0);
    float *sB = sm, *sq = sB + C * LD, *sk = sq + C * LD, *low = sk + C * LD;  // [C][LD] each, [C][rank]
    for (int i = tid; i < n * p.rank; i += 256) {
        const int t = i / p.rank, r = i - t * p.rank;
        low[i] = p.proj[(size_t)(t0 + t) * p.ldp + 2 * HD + 2 * HV + r];
    }
    __syncthreads();
    for (int i = tid; i < C * LD; i += 256) {
        const int t = i / LD, d = i - t * LD;
        float l = 0.f, q = 0.f, k = 0.f;
        if (t < n && d < dim) {
            const float* row = p.proj + (size_t)(t0 + t) * p.ldp + h * dim + d;
            q = row[0] * p.qscale;
            k = row[HD];
            l = log_decay(p, low + t * p.rank, h * dim + d);
        }
        sB[i] = l;
        sq[i] = q;
        sk[i] = k;
    }
    __syncthreads();
    for (int d = tid; d < dim; d += 256) {
        float s = 0.f;
        for (int t = 0; t < C; ++t) {
            s += sB[t * LD + d];
            sB[t * LD + d] = s;
        }
        b.decay[((size_t)ch * p.heads + h) * dim + d] = expf(s);
    }
    __syncthreads();
    const float* end = sB + (C - 1) * LD;
    for (int i = tid; i < n * dim; i += 256) {
        const int t = i / dim, d = i - t * dim;
        const float B = sB[t * LD + d];
        const size_t at = (size_t)(t0 + t) * HD + h * dim + d;
        b.qd[at] = sq[t * LD + d] * expf(B);
        b.kd[at] = sk[t * LD + d] * expf(end[d] - B);
    }
    float* A = b.weights + ((size_t)ch * p.heads + h) * C * C;
    const int nsub = C / kSub;
    // pairs inside a sub-block: a warp per pair (t >= s)
    const int warp = tid >> 5, lane = tid & 31;
    for (int i = tid; i < C * C; i += 256) {
        const int t = i / C, s = i - t * C;
        if (s > t) A[i] = 0.f;
    }
    for (int sub = 0; sub < nsub; ++sub) {
        const int base = sub * kSub;
        if (base >= n) break;
        for (int pr = warp; pr < kSub * (kSub + 1) / 2; pr += 8) {
            int t = 0, left = pr;
            while (left > t) left -= ++t;
            const float *qt = sq + (base + t) * LD, *ks = sk + (base + left) * LD, *Bt = sB + (base + t) * LD, *Bs = sB + (base + left) * LD;
            float a = 0.f;
            for (int d = lane; d < dim; d += 32) a = fmaf(qt[d] * ks[d], expf(Bt[d] - Bs[d]), a);
            a = lb_warp_sumf(a);
            if (lane == 0) A[(base + t) * C + base + left] = a;
        }
    }
    // pairs of different sub-blocks: queries of sub-block i decayed from its border, keys of the earlier ones decayed to it
    for (int i = 1; i < nsub; ++i) {
        const int base = i * kSub;
        if (base >= n) break;
        const float* ref = sB + (base - 1) * LD;
        __syncthreads();
        // in place: the queries of this sub-block are not used again; the keys move from border to border
        for (int e = tid; e < kSub * dim; e += 256) {
            const int t = base + e / dim, d = e % dim;
            sq[t * LD + d] *= expf(sB[t * LD + d] - ref[d]);
        }
        const float* prev = sB + (base - kSub - 1) * LD;  // border of the sub-block before
        for (int e = tid; e < base * dim; e += 256) {
            const int s = e / dim, d = e % dim;
            const float from = s < base - kSub ? prev[d] : sB[s * LD + d];
            sk[s * LD + d] *= expf(ref[d] - from);
        }
        __syncthreads();
        // 16 x base outputs, 2 x 2 per thread
        for (int o = tid; o < (kSub / 2) * (base / 2); o += 256) {
            const int t = base + 2 * (o / (base / 2)), s = 2 * (o % (base / 2));
            const float *q0 = sq + t * LD, *q1 = q0 + LD, *k0 = sk + s * LD, *k1 = k0 + LD;
            float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
            for (int d = 0; d < dim; d += 4) {  // (columns dim .. LD are zero)
                const float4 x = *reinterpret_cast<const float4*>(q0 + d), y = *reinterpret_cast<const float4*>(q1 + d);
                const float4 u = *reinterpret_cast<const float4*>(k0 + d), w = *reinterpret_cast<const float4*>(k1 + d);
                a00 = fmaf(x.x, u.x, fmaf(x.y, u.y, fmaf(x.z, u.z, fmaf(x.w, u.w, a00))));
                a01 = fmaf(x.x, w.x, fmaf(x.y, w.y, fmaf(x.z, w.z, fmaf(x.w, w.w, a01))));
                a10 = fmaf(y.x, u.x, fmaf(y.y, u.y, fmaf(y.z, u.z, fmaf(y.w, u.w, a10))));
                a11 = fmaf(y.x, w.x, fmaf(y.y, w.y, fmaf(y.z, w.z, fmaf(y.w, w.w, a11))));
            }
            A[t * C + s] = a00;
            A[t * C + s + 1] = a01;
            A[(t + 1) * C + s] = a10;
            A[(t + 1) * C + s + 1] = a11;
        }
    }
}

// 64 x 64 output tiles of products of float matrices: 256 threads, 4 x 4 each
constexpr int kTile = 64, kTileLd = 68;

__device__ __forceinline__ void tile_fma(const float (*sa)[kTileLd], const float (*sb)[kTileLd], int n, int ty, int tx, float (*acc)[4]) {
#pragma unroll 8
    for (int k = 0; k < n; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(&sa[k][ty * 4]), b = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
        const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
}

// what a chunk adds to the state: CTA = (64 channels x 64 value columns, head, chunk)
__global__ void __launch_bounds__(256) lb_gla_state_kernel(const LbGla p, const LbGlaBlock b, int T, int dtiles) {
    __shared__ __align__(16) float sa[32][kTileLd], sb[32][kTileLd];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int d0 = (blockIdx.x % dtiles) * kTile, v0 = (blockIdx.x / dtiles) * kTile, h = blockIdx.y, ch = blockIdx.z, tid = threadIdx.x;
    const int HD = p.heads * p.dim, t0 = ch * b.C, n = min(b.C, T - t0), ty = tid >> 4, tx = tid & 15;
    float acc[4][4] = {};
    for (int s0 = 0; s0 < n; s0 += 32) {
        __syncthreads();
        for (int i = tid; i < 32 * kTile; i += 256) {
            const int t = i >> 6, c = i & 63, tt = s0 + t;
            const bool ok = tt < n;
            sa[t][c] = ok && d0 + c < p.dim ? b.kd[(size_t)(t0 + tt) * HD + h * p.dim + d0 + c] : 0.f;
            sb[t][c] = ok && v0 + c < p.vdim ? p.proj[(size_t)(t0 + tt) * p.ldp + 2 * HD + h * p.vdim + v0 + c] : 0.f;
        }
        __syncthreads();
        tile_fma(sa, sb, 32, ty, tx, acc);
    }
    float* out = b.states + ((size_t)ch * p.heads + h) * p.dim * p.vdim;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int d = d0 + ty * 4 + i, v = v0 + tx * 4 + j;
            if (d < p.dim && v < p.vdim) out[(size_t)d * p.vdim + v] = acc[i][j];
        }
}

// what the chunks add -> the state in front of every chunk, in place; the last state becomes the sequence's
__global__ void __launch_bounds__(256) lb_gla_scan_kernel(const LbGla p, const LbGlaBlock b, int chunks, int fresh) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const size_t all = (size_t)p.heads * p.dim * p.vdim, i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= all) return;
    const size_t hd = i / p.vdim;
    float s = fresh ? 0.f : p.state[i];
    constexpr int U = 8;
    for (int c0 = 0; c0 < chunks; c0 += U) {
        float add[U], dec[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = c0 + u;
            add[u] = c < chunks ? b.states[(size_t)c * all + i] : 0.f;
            dec[u] = c < chunks ? b.decay[(size_t)c * p.heads * p.dim + hd] : 1.f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < chunks) b.states[(size_t)(c0 + u) * all + i] = s;
            s = fmaf(dec[u], s, add[u]);
        }
    }
    p.state[i] = s;
}

// outputs: CTA = (64 value columns, head, chunk): (scaled queries | weights) times (state | values)
__global__ void __launch_bounds__(256) lb_gla_out_kernel(const LbGla p, const LbGlaBlock b, int T) {
    __shared__ __align__(16) float sa[32][kTileLd], sb[32][kTileLd];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int v0 = blockIdx.x * kTile, h = blockIdx.y, ch = blockIdx.z, tid = threadIdx.x, C = b.C;
    const int HD = p.heads * p.dim, t0 = ch * C, n = min(C, T - t0), ty = tid >> 4, tx = tid & 15;
    const float* S = b.states + ((size_t)ch * p.heads + h) * p.dim * p.vdim;
    const float* A = b.weights + ((size_t)ch * p.heads + h) * C * C;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < p.dim; k0 += 32) {
        __syncthreads();
        for (int i = tid; i < 32 * kTile; i += 256) {
            const int t = i >> 5, k = i & 31;
            sa[k][t] = t < n && k0 + k < p.dim ? b.qd[(size_t)(t0 + t) * HD + h * p.dim + k0 + k] : 0.f;
            const int kk = i >> 6, c = i & 63;
            sb[kk][c] = k0 + kk < p.dim && v0 + c < p.vdim ? S[(size_t)(k0 + kk) * p.vdim + v0 + c] : 0.f;
        }
        __syncthreads();
        tile_fma(sa, sb, 32, ty, tx, acc);
    }
    for (int s0 = 0; s0 < n; s0 += 32) {
        __syncthreads();
        for (int i = tid; i < 32 * kTile; i += 256) {
            const int t = i >> 5, s = i & 31;
            sa[s][t] = t < n && s0 + s < n ? A[t * C + s0 + s] : 0.f;
            const int kk = i >> 6, c = i & 63;
            sb[kk][c] = s0 + kk < n && v0 + c < p.vdim ? p.proj[(size_t)(t0 + s0 + kk) * p.ldp + 2 * HD + h * p.vdim + v0 + c] : 0.f;
        }
        __syncthreads();
        tile_fma(sa, sb, 32, ty, tx, acc);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty * 4 + i;
        if (t >= n) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int v = v0 + tx * 4 + j;
            if (v < p.vdim) p.o[(size_t)(t0 + t) * p.ldo + h * p.vdim + v] = acc[i][j];
        }
    }
}

size_t prep_smem(int C, int dim, int rank) { return ((size_t)3 * C * (lb_round_up(dim, 4) + 4) + (size_t)C * rank) * sizeof(float); }

}  // namespace

int lb_gla_chunk(int dim, int rank) {
    for (int C = 64; C >= kSub; C /= 2)
        if (prep_smem(C, dim, rank) <= 200 * 1024) return C;
    return 0;
}

int lb_gla_step(loom_b200_ctx* ctx, const LbGla& p, const int* pos, int lane0, int M) {
    const size_t smem = (size_t)(3 * p.dim + p.rank) * sizeof(float);
    LB_REQUIRE(ctx, smem <= 40 * 1024, "gla: %d key channels, decay rank %d", p.dim, p.rank);
    LB_LAUNCH(ctx, lb_gla_step_kernel, dim3(lb_ceil_div(p.vdim, 32), p.heads, M), dim3(256), smem, p, pos, lane0);
    return 0;
}

int lb_gla_block(loom_b200_ctx* ctx, const LbGla& p, const LbGlaBlock& bin, int T, int pos0) {
    LbGlaBlock b = bin;
    b.C = lb_gla_chunk(p.dim, p.rank);
    LB_REQUIRE(ctx, b.C > 0, "gla: %d key channels, decay rank %d", p.dim, p.rank);
    const int chunks = lb_ceil_div(T, b.C), fresh = pos0 == 0 ? 1 : 0;
    LB_BIG_SMEM(ctx, lb_gla_prep_kernel, 200 * 1024);
    LB_LAUNCH(ctx, lb_gla_prep_kernel, dim3(chunks, p.heads), dim3(256), prep_smem(b.C, p.dim, p.rank), p, b, T);
    const int dt = lb_ceil_div(p.dim, kTile), vt = lb_ceil_div(p.vdim, kTile);
    LB_LAUNCH(ctx, lb_gla_state_kernel, dim3(dt * vt, p.heads, chunks), dim3(256), 0, p, b, T, dt);
    const size_t all = (size_t)p.heads * p.dim * p.vdim;
    LB_LAUNCH(ctx, lb_gla_scan_kernel, dim3((unsigned)((all + 255) / 256)), dim3(256), 0, p, b, chunks, fresh);
    LB_LAUNCH(ctx, lb_gla_out_kernel, dim3(vt, p.heads, chunks), dim3(256), 0, p, b, T);
    return 0;
}
