// matrix_memory.cu -- matrix memory with exponential gates (mLSTM): the one-token step and the token block.
//
//   m_t = max(f_t + m_(t-1), i_t),  S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,  n_t likewise with k_t alone,
//   o_t = S_t^T q_t / (max(|n_t.q_t|, e^(-m_t)) + 1e-6),   m = 0, S = 0, n = 0 in front of a sequence
//
// A block of tokens is cut into chunks of C.  With F_t the sum of f inside a chunk, m, S and n in front of it,
//   S_t^T q_t = e^(F_t + m - m_t) S^T q_t + sum_(s <= t) A_ts v_s,   A_ts = e^(F_t - F_s + i_s - m_t) q_t.k_s
// and n_t.q_t is the same with ones for v.  The maxima are a scan of numbers (pairs (F, M): m -> max(m + F, M)), which every CTA
// repeats for the tokens in front of its chunk; after that chunks are independent but for the states, which gated_linear.cu's
// products carry.  No exponent but -m_t is ever positive; sums of f are 64-bit, everything else 32-bit floats.
#include "mixers.cuh"

namespace {

constexpr float kDenEps = 1e-6f;

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(__fdiv_rn(z, cap)); }
__device__ __forceinline__ void gates(const LbMemory& p, const float* row, int h, float& i, float& f) {
    const float* z = row + 2 * p.heads * (p.dim + p.vdim) + h;
    i = capped(z[0] + p.bias_i[h], p.cap);
    f = lb_log_sigmoidf(capped(z[p.heads] + p.bias_f[h], p.cap));
}

// ---- one token of each of M sequences: CTA = (32 value columns, head, sequence); warps split the key channels -----------
__global__ void __launch_bounds__(256) lb_memory_step_kernel(const LbMemory p, const int* pos_of, int lane0) {
    extern __shared__ float sm[];
    __shared__ float part[8][32], red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.y, m = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, HD = p.heads * p.dim, pos = pos_of[m];
    float *sq = sm, *sk = sm + p.dim;
    const float* row = p.proj + (size_t)m * p.ldp;
    const int v = blockIdx.x * 32 + lane;
    const bool live = v < p.vdim, fresh = pos == 0;
    float* S = p.state + (((size_t)(lane0 + m) * p.heads + h) * p.dim) * p.vdim + v;
    float first[8];  // the first state rows of this warp are on their way while the gates are computed
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = warp + 8 * i;
        first[i] = live && !fresh && d < p.dim ? S[(size_t)d * p.vdim] : 0.f;
    }
    const int was = (pos + 1) & 1, now = pos & 1;
    const float vv = live ? row[2 * HD + h * p.vdim + v] : 0.f;
    float gi, gf;
    gates(p, row, h, gi, gf);
    const float m0 = fresh ? 0.f : p.top[((size_t)(lane0 + m) * 2 + was) * p.heads + h];
    const float mt = fmaxf(gf + m0, gi), keep = expf(gf + m0 - mt), put = expf(gi - mt);
    const float* nold = p.norm + (((size_t)(lane0 + m) * 2 + was) * p.heads + h) * p.dim;
    float* nnew = p.norm + (((size_t)(lane0 + m) * 2 + now) * p.heads + h) * p.dim;
    float den = 0.f;
    for (int d = tid; d < p.dim; d += 256) {
        const float q = row[h * p.dim + d] * p.qscale, k = row[HD + h * p.dim + d] * put;
        const float nn = fresh ? k : fmaf(keep, nold[d], k);
        sq[d] = q;
        sk[d] = k;
        den = fmaf(nn, q, den);
        if (blockIdx.x == 0) nnew[d] = nn;
    }
    if (blockIdx.x == 0 && tid == 0) p.top[((size_t)(lane0 + m) * 2 + now) * p.heads + h] = mt;
    den = lb_block_sumf(den, red);  // (its barriers also publish the rows)
    float acc = 0.f;
    auto row_step = [&](int d, float old) {
        const float s = fmaf(keep, old, sk[d] * vv);
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
        p.o[(size_t)m * p.ldo + h * p.vdim + v] = __fdiv_rn(o, fmaxf(fabsf(den), expf(-mt)) + kDenEps);
    }
}

// ---- token blocks ------------------------------------------------------------------------------------------------------

__host__ __device__ inline int lead(int dim) { return lb_round_up(dim, 4) + 4; }

// tokens in a row: the sum of their f and the largest i + sum of the f behind it; first a, then b
struct Run {
    double F;
    float M;
};
__device__ __forceinline__ Run join(const Run& a, const Run& b) { return {a.F + b.F, fmaxf((float)(a.M + b.F), b.M)}; }

// log gates of every token, [heads][T]
__global__ void __launch_bounds__(256) lb_memory_gates_kernel(const LbMemory p, const LbMemoryBlock b, int T) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int i = blockIdx.x * 256 + threadIdx.x;
    if (i >= T * p.heads) return;
    const int t = i / p.heads, h = i - t * p.heads;
    float gi, gf;
    gates(p, p.proj + (size_t)t * p.ldp, h, gi, gf);
    b.gate_i[(size_t)h * T + t] = gi;
    b.gate_f[(size_t)h * T + t] = gf;
}

__device__ __forceinline__ void put4(float* row, int d, int n, bool vec, const float* f) {
    if (vec) {
        *reinterpret_cast<float4*>(row + d) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
#pragma unroll
        for (int e = 0; e < 4; ++e)
            if (d + e < n) row[d + e] = f[e];
    }
}

// CTA = (chunk, head): maxima, weights, and the operands of the products over chunks
template <int C>
__global__ void __launch_bounds__(256, 3) lb_memory_prep_kernel(const LbMemory p, const LbMemoryBlock b, int T, int pos0, bool vec) {
    extern __shared__ __align__(16) float sm[];
    __shared__ Run s_run[8];
    __shared__ double s_F[C];
    __shared__ float s_i[C], s_f[C], s_m[C], s_keep[C], s_end[C], s_m0;
    constexpr int NI = C / 16, LC = C + 4;
    const int ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, dim = p.dim, LD = lead(dim);
    const int HD = p.heads * dim, t0 = ch * C, n = min(C, T - t0), D4 = lb_round_up(dim, 4) / 4;
    float *sk = sm, *sq = sk + C * LD, *sa = sq;  // sa [C][LC]: the weights, in place of the queries
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const float *gi = b.gate_i + (size_t)h * T, *gf = b.gate_f + (size_t)h * T;
    for (int i = tid; i < C * D4; i += 256) {
        const int t = i / D4, d = (i - t * D4) * 4;
        float q[4] = {0.f, 0.f, 0.f, 0.f}, k[4] = {0.f, 0.f, 0.f, 0.f};
        if (t < n) {
            const float* row = p.proj + (size_t)(t0 + t) * p.ldp + h * dim;
            lb_load_cols<4>(row, d, dim, vec, q);
            lb_load_cols<4>(row + HD, d, dim, vec, k);
        }
        *reinterpret_cast<float4*>(sq + t * LD + d) = make_float4(q[0] * p.qscale, q[1] * p.qscale, q[2] * p.qscale, q[3] * p.qscale);
        *reinterpret_cast<float4*>(sk + t * LD + d) = make_float4(k[0], k[1], k[2], k[3]);
    }
    if (tid < C) {
        s_i[tid] = tid < n ? gi[t0 + tid] : -INFINITY;
        s_f[tid] = tid < n ? gf[t0 + tid] : 0.f;
    }
    {
        const int per = lb_ceil_div(t0, 256);
        Run r = {0.0, -INFINITY};
        for (int t = tid * per; t < min(t0, (tid + 1) * per); ++t) r = join(r, {(double)gf[t], gi[t]});
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const Run right = {__shfl_down_sync(0xffffffffu, r.F, o), __shfl_down_sync(0xffffffffu, r.M, o)};
            r = join(r, right);  // (right where the lane is a multiple of 2 o)
        }
        if (lane == 0) s_run[warp] = r;
    }
    __syncthreads();
    if (tid == 0) {
        Run r = s_run[0];
        for (int w = 1; w < 8; ++w) r = join(r, s_run[w]);
        const float start = pos0 == 0 ? 0.f : p.top[(size_t)((pos0 + 1) & 1) * p.heads + h];
        float m = fmaxf((float)(start + r.F), r.M);
        double F = 0.0;
        s_m0 = m;
        for (int t = 0; t < C; ++t) {
            F += s_f[t];
            m = fmaxf(s_f[t] + m, s_i[t]);
            s_F[t] = F;
            s_m[t] = m;
        }
    }
    __syncthreads();
    if (tid < C) {
        s_keep[tid] = expf((float)(s_F[tid] + s_m0 - s_m[tid]));
        s_end[tid] = expf((float)(s_F[C - 1] - s_F[tid] + s_i[tid] - s_m[C - 1]));
        if (tid < n) b.tops[(size_t)(t0 + tid) * p.heads + h] = s_m[tid];
    }
    __syncthreads();
    {
        const int ty = tid >> 4, tx = tid & 15;
        float qk[NI][NI] = {};
        for (int d = 0; d < dim; d += 4) {  // (columns dim .. LD are zero)
            float4 q[NI], k[NI];
#pragma unroll
            for (int i = 0; i < NI; ++i) {
                q[i] = *reinterpret_cast<const float4*>(sq + (ty + 16 * i) * LD + d);
                k[i] = *reinterpret_cast<const float4*>(sk + (tx + 16 * i) * LD + d);
            }
#pragma unroll
            for (int i = 0; i < NI; ++i)
#pragma unroll
                for (int j = 0; j <= i; ++j) qk[i][j] = fmaf(q[i].x, k[j].x, fmaf(q[i].y, k[j].y, fmaf(q[i].z, k[j].z, fmaf(q[i].w, k[j].w, qk[i][j]))));
        }
        for (int i = tid; i < n * D4; i += 256) {  // queries decayed from the chunk's start
            const int t = i / D4, d = (i - t * D4) * 4;
            const float4 q = *reinterpret_cast<const float4*>(sq + t * LD + d);
            const float f[4] = {q.x * s_keep[t], q.y * s_keep[t], q.z * s_keep[t], q.w * s_keep[t]};
            put4(b.c.qd + (size_t)(t0 + t) * HD + h * dim, d, dim, vec, f);
        }
        __syncthreads();
        float* A = b.c.weights + ((size_t)ch * p.heads + h) * C * C;
#pragma unroll
        for (int i = 0; i < NI; ++i)
#pragma unroll
            for (int j = 0; j < NI; ++j) {
                const int t = ty + 16 * i, s = tx + 16 * j;
                float w = 0.f;
                if (j <= i && s <= t && t < n) w = qk[i][j] * expf((float)(s_F[t] - s_F[s] + s_i[s] - s_m[t]));
                sa[t * LC + s] = w;
                A[t * C + s] = w;
            }
    }
    __syncthreads();
    for (int t = warp; t < n; t += 8) {
        float s = 0.f;
        for (int x = lane; x < C; x += 32) s += sa[t * LC + x];
        s = lb_warp_sumf(s);
        if (lane == 0) b.sums[(size_t)(t0 + t) * p.heads + h] = s;
    }
    // keys decayed to the chunk's end
    const float over = s_keep[C - 1];
    for (int i = tid; i < n * D4; i += 256) {
        const int t = i / D4, d = (i - t * D4) * 4;
        const float4 k = *reinterpret_cast<const float4*>(sk + t * LD + d);
        const float f[4] = {k.x * s_end[t], k.y * s_end[t], k.z * s_end[t], k.w * s_end[t]};
        *reinterpret_cast<float4*>(sk + t * LD + d) = make_float4(f[0], f[1], f[2], f[3]);
        put4(b.c.kd + (size_t)(t0 + t) * HD + h * dim, d, dim, vec, f);
    }
    __syncthreads();
    for (int d = tid; d < dim; d += 256) {
        float s = 0.f;
#pragma unroll 8
        for (int t = 0; t < n; ++t) s += sk[t * LD + d];
        const size_t at = ((size_t)ch * p.heads + h) * dim + d;
        b.norms[at] = s;
        b.c.decay[at] = over;
    }
}

// the normaliser in front of every chunk; the last one and the last maximum become the sequence's
__global__ void __launch_bounds__(256) lb_memory_norms_kernel(const LbMemory p, const LbMemoryBlock b, int chunks, int T, int pos0) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int HD = p.heads * p.dim, i = blockIdx.x * 256 + threadIdx.x;
    const int was = (pos0 + 1) & 1, now = (pos0 + T - 1) & 1;
    if (i < p.heads) p.top[(size_t)now * p.heads + i] = b.tops[(size_t)(T - 1) * p.heads + i];
    if (i >= HD) return;
    float s = pos0 == 0 ? 0.f : p.norm[(size_t)was * HD + i];
    constexpr int U = 8;
    for (int c0 = 0; c0 < chunks; c0 += U) {
        float add[U], dec[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            add[u] = c0 + u < chunks ? b.norms[(size_t)(c0 + u) * HD + i] : 0.f;
            dec[u] = c0 + u < chunks ? b.c.decay[(size_t)(c0 + u) * HD + i] : 1.f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < chunks) b.norms[(size_t)(c0 + u) * HD + i] = s;
            s = fmaf(dec[u], s, add[u]);
        }
    }
    p.norm[(size_t)now * HD + i] = s;
}

// a warp per (token, head)
__global__ void __launch_bounds__(256) lb_memory_scale_kernel(const LbMemory p, const LbMemoryBlock b, int T) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (i >= T * p.heads) return;
    const int t = i / p.heads, h = i - t * p.heads;
    const float *q = b.c.qd + (size_t)i * p.dim, *nn = b.norms + ((size_t)(t / b.c.C) * p.heads + h) * p.dim;
    float d = 0.f;
    for (int k = lane; k < p.dim; k += 32) d = fmaf(q[k], nn[k], d);
    d = lb_warp_sumf(d) + b.sums[i];
    if (lane == 0) b.scale[i] = __fdiv_rn(1.f, fmaxf(fabsf(d), expf(-b.tops[i])) + kDenEps);
}

size_t prep_smem(int C, int dim) {
    const size_t q = lead(dim) > C + 4 ? lead(dim) : C + 4;
    return (size_t)C * (lead(dim) + q) * sizeof(float);
}

template <int C>
int launch_prep(loom_b200_ctx* ctx, const LbMemory& p, const LbMemoryBlock& b, int T, int pos0) {
    LB_BIG_SMEM(ctx, lb_memory_prep_kernel<C>, 200 * 1024);
    const bool vec = p.dim % 4 == 0 && lb_vec_rows(p.proj, p.ldp);
    LB_LAUNCH(ctx, lb_memory_prep_kernel<C>, dim3(lb_ceil_div(T, C), p.heads), dim3(256), prep_smem(C, p.dim), p, b, T, pos0, vec);
    return 0;
}

}  // namespace

int lb_memory_chunk(int dim) {
    for (int C = 64; C >= 16; C /= 2)
        if (prep_smem(C, dim) <= 200 * 1024) return C;
    return 0;
}

int lb_memory_step(loom_b200_ctx* ctx, const LbMemory& p, const int* pos, int lane0, int M) {
    const size_t smem = (size_t)2 * p.dim * sizeof(float);
    LB_REQUIRE(ctx, smem <= 40 * 1024, "matrix memory: %d key channels", p.dim);
    LB_LAUNCH(ctx, lb_memory_step_kernel, dim3(lb_ceil_div(p.vdim, 32), p.heads, M), dim3(256), smem, p, pos, lane0);
    return 0;
}

int lb_memory_block(loom_b200_ctx* ctx, const LbMemory& p, const LbMemoryBlock& bin, int T, int pos0) {
    LbMemoryBlock b = bin;
    b.c.C = lb_memory_chunk(p.dim);
    LB_REQUIRE(ctx, b.c.C > 0, "matrix memory: %d key channels", p.dim);
    b.c.heads = p.heads;
    b.c.dim = p.dim;
    b.c.vdim = p.vdim;
    b.c.v = p.proj + 2 * p.heads * p.dim;
    b.c.ldv = p.ldp;
    b.c.state = p.state;
    b.c.o = p.o;
    b.c.ldo = p.ldo;
    const int chunks = lb_ceil_div(T, b.c.C);
    LB_LAUNCH(ctx, lb_memory_gates_kernel, dim3(lb_ceil_div(T * p.heads, 256)), dim3(256), 0, p, b, T);
    int rc = b.c.C == 64 ? launch_prep<64>(ctx, p, b, T, pos0) : b.c.C == 32 ? launch_prep<32>(ctx, p, b, T, pos0) : launch_prep<16>(ctx, p, b, T, pos0);
    if (rc) return rc;
    if ((rc = lb_chunk_states(ctx, b.c, T))) return rc;
    if ((rc = lb_chunk_scan(ctx, b.c, T, pos0 == 0))) return rc;
    LB_LAUNCH(ctx, lb_memory_norms_kernel, dim3(lb_ceil_div(p.heads * p.dim, 256)), dim3(256), 0, p, b, chunks, T, pos0);
    if ((rc = lb_chunk_out(ctx, b.c, T))) return rc;
    LB_LAUNCH(ctx, lb_memory_scale_kernel, dim3(lb_ceil_div(T * p.heads, 8)), dim3(256), 0, p, b, T);
    return 0;
}
