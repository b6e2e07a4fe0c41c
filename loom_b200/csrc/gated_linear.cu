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

constexpr int kPrepThreads = 256;
constexpr int kRankBlock = 16;

// sums of sixteen values over a warp: afterwards lane l (and l + 16) holds the sum of value bit-reversed(l & 15)
__device__ __forceinline__ float warp_sum16(float* v, int lane) {
#pragma unroll
    for (int w = 8, bit = 1; w >= 1; w >>= 1, bit <<= 1) {
        const bool up = lane & bit;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
            if (i >= w) break;
            const float send = up ? v[i] : v[i + w], keep = up ? v[i + w] : v[i];
            v[i] = keep + __shfl_xor_sync(0xffffffffu, send, bit);
        }
    }
    return v[0] + __shfl_xor_sync(0xffffffffu, v[0], 16);
}

// CTA = (chunk, head): decays, the scaled queries and keys and the chunk's token-by-token weights
__global__ void __launch_bounds__(kPrepThreads, 2) lb_gla_prep_kernel(const LbGla p, const LbChunks b, int T) {
    extern __shared__ __align__(16) float sm[];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int C = b.C, ch = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, dim = p.dim, LD = lb_round_up(dim, 4) + 4, RP = lb_round_up(p.rank, kRankBlock);
    const int HD = p.heads * dim, HV = p.heads * p.vdim, t0 = ch * C, n = min(C, T - t0), nsub = C / kSub;
    float *sB = sm, *sq = sB + C * LD, *sk = sq + C * LD, *low = sk + C * LD;  // [C][LD] each, [C][RP]; later the factors between sub-blocks
    for (int i = tid; i < C * RP; i += kPrepThreads) {
        const int t = i / RP, r = i - t * RP;
        low[i] = t < n && r < p.rank ? p.proj[(size_t)(t0 + t) * p.ldp + 2 * HD + 2 * HV + r] : 0.f;
    }
    for (int i = tid; i < C * LD; i += kPrepThreads) {
        const int t = i / LD, d = i - t * LD;
        const float* row = p.proj + (size_t)(t0 + t) * p.ldp + h * dim + d;
        const bool ok = t < n && d < dim;
        sq[i] = ok ? row[0] * p.qscale : 0.f;
        sk[i] = ok ? row[HD] : 0.f;
    }
    __syncthreads();
    // threads (channel, part of the chunk's tokens)
    int DS = 32;
    while (DS < dim && DS < kPrepThreads) DS *= 2;
    const int parts = kPrepThreads / DS, part = tid / DS, per = C / parts, ta = part * per;
    for (int d = tid % DS; d < dim; d += DS) {
        const float bias = p.a2b[h * dim + d];
        for (int rb = 0; rb < p.rank; rb += kRankBlock) {
            float w[kRankBlock];
#pragma unroll
            for (int r = 0; r < kRankBlock; ++r) w[r] = rb + r < p.rank ? p.a2t[(size_t)(rb + r) * HD + h * dim + d] : 0.f;
            const bool done = rb + kRankBlock >= p.rank;
            for (int t = ta; t < ta + per; ++t) {
                float z = rb == 0 ? bias : sB[t * LD + d];
                const float4* x = reinterpret_cast<const float4*>(low + t * RP + rb);
#pragma unroll
                for (int r = 0; r < kRankBlock / 4; ++r) {
                    const float4 v = x[r];
                    z = fmaf(w[4 * r], v.x, fmaf(w[4 * r + 1], v.y, fmaf(w[4 * r + 2], v.z, fmaf(w[4 * r + 3], v.w, z))));
                }
                if (done) {
                    const float l = t < n ? lb_log_sigmoidf(z) * p.inv_tau : 0.f;
                    if (t < n) b.kd[(size_t)(t0 + t) * HD + h * dim + d] = l;  // kept here while the decays themselves are needed
                    z = expf(l);
                }
                sB[t * LD + d] = z;
            }
        }
    }
    __syncthreads();
    float* A = b.weights + ((size_t)ch * p.heads + h) * C * C;
    for (int i = tid; i < C * C; i += kPrepThreads) {
        const int t = i / C, s = i - t * C;
        if (s > t) A[i] = 0.f;
    }
    // pairs inside a sub-block: the product of the decays between the two tokens grows step by step in a register.  Lanes split the
    // channels (128 at a time), the warps of a sub-block split its keys
    const int warp = tid >> 5, lane = tid & 31;
    const int wps = 8 / nsub > 0 ? 8 / nsub : 1;  // warps per sub-block
    for (int sub = warp / wps; sub < nsub; sub += 8 / wps) {
        const int base = sub * kSub;
        if (base >= n) break;
        for (int d0 = 0; d0 < dim; d0 += 128) {
            float a[kSub][4];
#pragma unroll
            for (int t = 0; t < kSub; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) a[t][e] = d0 + 32 * e + lane < dim ? sB[(base + t) * LD + d0 + 32 * e + lane] : 0.f;
            for (int s = warp % wps; s < kSub; s += wps) {
                float f[4], v[kSub];
#pragma unroll
                for (int e = 0; e < 4; ++e) f[e] = d0 + 32 * e + lane < dim ? sk[(base + s) * LD + d0 + 32 * e + lane] : 0.f;
#pragma unroll
                for (int t = 0; t < kSub; ++t) {
                    v[t] = 0.f;
                    if (t >= s) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            if (t > s) f[e] *= a[t][e];
                            if (d0 + 32 * e < dim) v[t] = fmaf(d0 + 32 * e + lane < dim ? sq[(base + t) * LD + d0 + 32 * e + lane] : 0.f, f[e], v[t]);
                        }
                    }
                }
                const float sum = warp_sum16(v, lane);
                const int t = ((lane & 1) << 3) | ((lane & 2) << 1) | ((lane & 4) >> 1) | ((lane & 8) >> 3);
                if (lane < 16 && t >= s) {
                    float* out = A + (base + t) * C + base + s;
                    *out = d0 == 0 ? sum : *out + sum;
                }
            }
        }
    }
    __syncthreads();
    // running sums of the log decays
    for (int d = tid % DS; d < dim; d += DS) {
        float s = 0.f;
        for (int t = ta; t < ta + per; ++t) {
            s += t < n ? b.kd[(size_t)(t0 + t) * HD + h * dim + d] : 0.f;
            sB[t * LD + d] = s;
        }
    }
    __syncthreads();
    if (parts > 1) {  // (then a thread has one channel)
        const int d = tid % DS;
        float off = 0.f;
        if (d < dim)
            for (int q = 0; q < part; ++q) off += sB[(q * per + per - 1) * LD + d];
        __syncthreads();
        if (d < dim && part > 0)
            for (int t = ta; t < ta + per; ++t) sB[t * LD + d] += off;
        __syncthreads();
    }
    const float* end = sB + (C - 1) * LD;
    for (int d = tid; d < dim; d += kPrepThreads) b.decay[((size_t)ch * p.heads + h) * dim + d] = expf(end[d]);
    // outputs, and in place: queries decayed from the border in front of their sub-block, keys to the end of theirs
    for (int i = tid; i < n * dim; i += kPrepThreads) {
        const int t = i / dim, d = i - t * dim, border = (t / kSub) * kSub - 1;
        const float B = sB[t * LD + d], q = sq[t * LD + d], k = sk[t * LD + d];
        const size_t at = (size_t)(t0 + t) * HD + h * dim + d;
        b.qd[at] = q * expf(B);
        b.kd[at] = k * expf(end[d] - B);
        if (border >= 0) sq[t * LD + d] = q * expf(B - sB[border * LD + d]);
        sk[t * LD + d] = k * expf(sB[(border + kSub) * LD + d] - B);
    }
    float* between = low;  // [(i, j) with i > j + 1][LD]: from the end of sub-block j to the border in front of sub-block i
    const int nb = (nsub - 1) * (nsub - 2) / 2;
    for (int x = tid; x < nb * LD; x += kPrepThreads) {
        const int d = x % LD;
        int i = 2, j = x / LD;
        while (j > i - 2) j -= i++ - 1;
        between[x] = d < dim ? expf(sB[(i * kSub - 1) * LD + d] - sB[(j * kSub + kSub - 1) * LD + d]) : 0.f;
    }
    __syncthreads();
    // pairs of different sub-blocks, 2 x 2 per thread
    constexpr int kItems = (kSub / 2) * (kSub / 2);
    for (int x = tid; x < nsub * (nsub - 1) / 2 * kItems; x += kPrepThreads) {
        int i = 1, j = x / kItems;
        while (j > i - 1) j -= i++;
        if (i * kSub >= n) continue;
        const int o = x % kItems, t = i * kSub + 2 * (o / (kSub / 2)), s = j * kSub + 2 * (o % (kSub / 2));
        const float *q0 = sq + t * LD, *q1 = q0 + LD, *k0 = sk + s * LD, *k1 = k0 + LD;
        const float* f = i - j > 1 ? between + ((i - 1) * (i - 2) / 2 + j) * LD : nullptr;
        float a00 = 0.f, a01 = 0.f, a10 = 0.f, a11 = 0.f;
        for (int d = 0; d < dim; d += 4) {  // (columns dim .. LD are zero)
            const float4 u = *reinterpret_cast<const float4*>(q0 + d), w = *reinterpret_cast<const float4*>(q1 + d);
            float4 y = *reinterpret_cast<const float4*>(k0 + d), z = *reinterpret_cast<const float4*>(k1 + d);
            if (f) {
                const float4 g = *reinterpret_cast<const float4*>(f + d);
                y = make_float4(y.x * g.x, y.y * g.y, y.z * g.z, y.w * g.w);
                z = make_float4(z.x * g.x, z.y * g.y, z.z * g.z, z.w * g.w);
            }
            a00 = fmaf(u.x, y.x, fmaf(u.y, y.y, fmaf(u.z, y.z, fmaf(u.w, y.w, a00))));
            a01 = fmaf(u.x, z.x, fmaf(u.y, z.y, fmaf(u.z, z.z, fmaf(u.w, z.w, a01))));
            a10 = fmaf(w.x, y.x, fmaf(w.y, y.y, fmaf(w.z, y.z, fmaf(w.w, y.w, a10))));
            a11 = fmaf(w.x, z.x, fmaf(w.y, z.y, fmaf(w.z, z.z, fmaf(w.w, z.w, a11))));
        }
        A[t * C + s] = a00;
        A[t * C + s + 1] = a01;
        A[(t + 1) * C + s] = a10;
        A[(t + 1) * C + s + 1] = a11;
    }
}

// 64 x 64 output tiles of products of float matrices: 128 threads, 8 x 4 each
constexpr int kTile = 64, kTileLd = 68, kTileK = 32, kTileThreads = 128;

__device__ __forceinline__ void tile_fma(const float (*sa)[kTileLd], const float (*sb)[kTileLd], int ty, int tx, float (*acc)[4]) {
#pragma unroll 8
    for (int k = 0; k < kTileK; ++k) {
        const float4 a = *reinterpret_cast<const float4*>(&sa[k][ty * 8]), a2 = *reinterpret_cast<const float4*>(&sa[k][ty * 8 + 4]);
        const float4 b = *reinterpret_cast<const float4*>(&sb[k][tx * 4]);
        const float av[8] = {a.x, a.y, a.z, a.w, a2.x, a2.y, a2.z, a2.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
        for (int i = 0; i < 8; ++i)
#pragma unroll
            for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
}
// rows k0 .. of a row-major matrix (nk of them exist), columns c0 .. (nc exist)
__device__ __forceinline__ void tile_rows(float (*s)[kTileLd], const float* m, size_t ld, int nk, int c0, int nc, bool vec) {
    for (int i = threadIdx.x; i < kTileK * kTile / 4; i += kTileThreads) {
        const int k = i >> 4, c = (i & 15) * 4;
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (k < nk) lb_load_cols<4>(m + (size_t)k * ld, c0 + c, nc, vec, f);
        *reinterpret_cast<float4*>(&s[k][c]) = make_float4(f[0], f[1], f[2], f[3]);
    }
}
// the same transposed: s[k][row] = m[row][k0 + k]
__device__ __forceinline__ void tile_cols(float (*s)[kTileLd], const float* m, size_t ld, int nr, int k0, int nk, bool vec) {
    for (int i = threadIdx.x; i < kTile * kTileK / 4; i += kTileThreads) {
        const int r = i & 63, k = (i >> 6) * 4;
        float f[4] = {0.f, 0.f, 0.f, 0.f};
        if (r < nr) lb_load_cols<4>(m + (size_t)r * ld, k0 + k, nk, vec, f);
#pragma unroll
        for (int e = 0; e < 4; ++e) s[k + e][r] = f[e];
    }
}

// what a chunk adds to the state: CTA = (64 channels x 64 value columns, head, chunk)
__global__ void __launch_bounds__(kTileThreads) lb_chunk_state_kernel(const LbChunks b, int T, int dtiles, bool vec) {
    __shared__ __align__(16) float sa[kTileK][kTileLd], sb[kTileK][kTileLd];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int d0 = (blockIdx.x % dtiles) * kTile, v0 = (blockIdx.x / dtiles) * kTile, h = blockIdx.y, ch = blockIdx.z, tid = threadIdx.x;
    const int HD = b.heads * b.dim, t0 = ch * b.C, n = min(b.C, T - t0), ty = tid >> 4, tx = tid & 15;
    float acc[8][4] = {};
    for (int s0 = 0; s0 < n; s0 += kTileK) {
        __syncthreads();
        tile_rows(sa, b.kd + (size_t)(t0 + s0) * HD + h * b.dim, HD, n - s0, d0, b.dim, vec);
        tile_rows(sb, b.v + (size_t)(t0 + s0) * b.ldv + h * b.vdim, b.ldv, n - s0, v0, b.vdim, vec);
        __syncthreads();
        tile_fma(sa, sb, ty, tx, acc);
    }
    float* out = b.states + ((size_t)ch * b.heads + h) * b.dim * b.vdim;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int d = d0 + ty * 8 + i, v = v0 + tx * 4;
        if (d >= b.dim) continue;
        if (vec && v + 4 <= b.vdim)
            *reinterpret_cast<float4*>(out + (size_t)d * b.vdim + v) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        else
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (v + j < b.vdim) out[(size_t)d * b.vdim + v + j] = acc[i][j];
    }
}

// what the chunks add -> the state in front of every chunk, in place; the last state becomes the sequence's
__global__ void __launch_bounds__(256) lb_chunk_scan_kernel(const LbChunks b, int chunks, int fresh) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const size_t all = (size_t)b.heads * b.dim * b.vdim, i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= all) return;
    const size_t hd = i / b.vdim;
    float s = fresh ? 0.f : b.state[i];
    constexpr int U = 8;
    for (int c0 = 0; c0 < chunks; c0 += U) {
        float add[U], dec[U];
#pragma unroll
        for (int u = 0; u < U; ++u) {
            const int c = c0 + u;
            add[u] = c < chunks ? b.states[(size_t)c * all + i] : 0.f;
            dec[u] = c < chunks ? b.decay[(size_t)c * b.heads * b.dim + hd] : 1.f;
        }
#pragma unroll
        for (int u = 0; u < U; ++u) {
            if (c0 + u < chunks) b.states[(size_t)(c0 + u) * all + i] = s;
            s = fmaf(dec[u], s, add[u]);
        }
    }
    b.state[i] = s;
}

// outputs: CTA = (64 value columns, head, chunk): (scaled queries | weights) times (state | values)
__global__ void __launch_bounds__(kTileThreads) lb_chunk_out_kernel(const LbChunks b, int T, bool vec) {
    __shared__ __align__(16) float sa[kTileK][kTileLd], sb[kTileK][kTileLd];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int v0 = blockIdx.x * kTile, h = blockIdx.y, ch = blockIdx.z, tid = threadIdx.x, C = b.C;
    const int HD = b.heads * b.dim, t0 = ch * C, n = min(C, T - t0), ty = tid >> 4, tx = tid & 15;
    const float* S = b.states + ((size_t)ch * b.heads + h) * b.dim * b.vdim;
    const float* A = b.weights + ((size_t)ch * b.heads + h) * C * C;
    float acc[8][4] = {};
    for (int k0 = 0; k0 < b.dim; k0 += kTileK) {
        __syncthreads();
        tile_cols(sa, b.qd + (size_t)t0 * HD + h * b.dim, HD, n, k0, b.dim, vec);
        tile_rows(sb, S + (size_t)k0 * b.vdim, b.vdim, b.dim - k0, v0, b.vdim, vec);
        __syncthreads();
        tile_fma(sa, sb, ty, tx, acc);
    }
    for (int s0 = 0; s0 < n; s0 += kTileK) {
        __syncthreads();
        tile_cols(sa, A, C, n, s0, n, true);
        tile_rows(sb, b.v + (size_t)(t0 + s0) * b.ldv + h * b.vdim, b.ldv, n - s0, v0, b.vdim, vec);
        __syncthreads();
        tile_fma(sa, sb, ty, tx, acc);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = ty * 8 + i, v = v0 + tx * 4;
        if (t >= n) continue;
        float* out = b.o + (size_t)(t0 + t) * b.ldo + h * b.vdim + v;
        if (vec && v + 4 <= b.vdim)
            *reinterpret_cast<float4*>(out) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
        else
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (v + j < b.vdim) out[j] = acc[i][j];
    }
}

size_t prep_smem(int C, int dim, int rank) {
    const size_t LD = lb_round_up(dim, 4) + 4, nsub = C / kSub, low = (size_t)C * lb_round_up(rank, kRankBlock), between = (nsub - 1) * (nsub > 2 ? nsub - 2 : 0) / 2 * LD;
    return (3 * C * LD + (low > between ? low : between)) * sizeof(float);
}

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

int lb_gla_block(loom_b200_ctx* ctx, const LbGla& p, const LbChunks& scratch, int T, int pos0) {
    LbChunks b = scratch;
    b.C = lb_gla_chunk(p.dim, p.rank);
    b.heads = p.heads;
    b.dim = p.dim;
    b.vdim = p.vdim;
    b.v = p.proj + 2 * p.heads * p.dim;
    b.ldv = p.ldp;
    b.state = p.state;
    b.o = p.o;
    b.ldo = p.ldo;
    LB_REQUIRE(ctx, b.C > 0, "gla: %d key channels, decay rank %d", p.dim, p.rank);
    LB_BIG_SMEM(ctx, lb_gla_prep_kernel, 200 * 1024);
    LB_LAUNCH(ctx, lb_gla_prep_kernel, dim3(lb_ceil_div(T, b.C), p.heads), dim3(kPrepThreads), prep_smem(b.C, p.dim, p.rank), p, b, T);
    if (int rc = lb_chunk_states(ctx, b, T)) return rc;
    if (int rc = lb_chunk_scan(ctx, b, T, pos0 == 0)) return rc;
    return lb_chunk_out(ctx, b, T);
}

int lb_chunk_states(loom_b200_ctx* ctx, const LbChunks& c, int T) {
    const bool vec = c.dim % 4 == 0 && c.vdim % 4 == 0 && lb_vec_rows(c.v, c.ldv);
    const int dt = lb_ceil_div(c.dim, kTile), vt = lb_ceil_div(c.vdim, kTile);
    LB_LAUNCH(ctx, lb_chunk_state_kernel, dim3(dt * vt, c.heads, lb_ceil_div(T, c.C)), dim3(kTileThreads), 0, c, T, dt, vec);
    return 0;
}

int lb_chunk_scan(loom_b200_ctx* ctx, const LbChunks& c, int T, bool fresh) {
    const size_t all = (size_t)c.heads * c.dim * c.vdim;
    LB_LAUNCH(ctx, lb_chunk_scan_kernel, dim3((unsigned)((all + 255) / 256)), dim3(256), 0, c, lb_ceil_div(T, c.C), fresh ? 1 : 0);
    return 0;
}

int lb_chunk_out(loom_b200_ctx* ctx, const LbChunks& c, int T) {
    const bool vec = c.dim % 4 == 0 && c.vdim % 4 == 0 && lb_vec_rows(c.v, c.ldv) && lb_vec_rows(c.o, c.ldo);
    LB_LAUNCH(ctx, lb_chunk_out_kernel, dim3(lb_ceil_div(c.vdim, kTile), c.heads, lb_ceil_div(T, c.C)), dim3(kTileThreads), 0, c, T, vec);
    return 0;
}
