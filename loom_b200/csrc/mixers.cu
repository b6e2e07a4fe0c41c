// mixers.cu -- kernels of mixers.cuh.
#include "mixers.cuh"

namespace {

// ---- embedding, norms, short convolution --------------------------------------------------------------------

template <typename WT>
__global__ void __launch_bounds__(256) lb_embed_norm_kernel(const WT* __restrict__ table, int vocab, int width, const int* tok, const float* gain,
                                                            float eps, float* __restrict__ x, int ldx) {
    __shared__ float red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = tok[blockIdx.x];
    float* out = x + (size_t)blockIdx.x * ldx;
    const bool ok = t >= 0 && t < vocab;
    const WT* row = table + (size_t)(ok ? t : 0) * width;
    float ss = 0.f;
    for (int k = threadIdx.x; k < width; k += blockDim.x) {
        const float v = ok ? (float)row[k] : 0.f;
        ss = fmaf(v, v, ss);
    }
    ss = lb_block_sumf(ss, red);
    const float r = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)width), eps))) * *gain;
    for (int k = threadIdx.x; k < width; k += blockDim.x) out[k] = ok ? (float)row[k] * r : 0.f;
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_embed_image_kernel(const uint8_t* __restrict__ img, int slices, int vocab, int width, const int* tok, float* __restrict__ x, int ldx) {
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = tok[blockIdx.x];
    const bool ok = t >= 0 && t < vocab;
    float* out = x + (size_t)blockIdx.x * ldx;
    for (int c = threadIdx.x; c < slices * 8; c += blockDim.x) {
        float f[C];
        lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(img + lb_img_chunk(ok ? t : 0, c, slices)), f);
        if ((c + 1) * C <= width) {  // (rows of x are padded to eight columns)
#pragma unroll
            for (int e = 0; e < C; e += 4) *reinterpret_cast<float4*>(out + c * C + e) = ok ? make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]) : make_float4(0.f, 0.f, 0.f, 0.f);
        } else {
#pragma unroll
            for (int e = 0; e < C; ++e)
                if (c * C + e < width) out[c * C + e] = ok ? f[e] : 0.f;
        }
    }
}

constexpr int kNormTokens = 8;  // tokens of a CTA
constexpr int kMaxTaps = 16;

__device__ __forceinline__ float row_rstd(const float* row, int width, float eps, int lane) {  // a warp per row
    float ss = 0.f;
    for (int k = lane; k < width; k += 32) ss = fmaf(row[k], row[k], ss);
    ss = lb_warp_sumf(ss);
    return __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)width), eps)));
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_norm_conv_kernel(const LbNormBlock p, bool vec) {
    constexpr int C = LbElem<WT>::kChunk;
    __shared__ float s_r[kNormTokens + kMaxTaps];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t0 = blockIdx.x * kNormTokens, t1 = min(p.T, t0 + kNormTokens);
    const int back = p.taps - 1;
    const float gain = *p.gain;
    for (int i = warp; i < t1 - t0 + back; i += 8) {
        const int t = t0 - back + i;
        if (t < 0) continue;
        const int src = p.row_idx ? p.row_idx[t] : t;
        const float r = row_rstd(p.x + (size_t)src * p.ldx, p.width, p.eps, lane) * gain;
        if (lane == 0) s_r[i] = r;
    }
    __syncthreads();
    const int chunks = p.slices * 8;
    for (int i = threadIdx.x; i < (t1 - t0) * chunks; i += blockDim.x) {
        const int tt = i / chunks, c = i - tt * chunks, t = t0 + tt, k0 = c * C;
        const int src = p.row_idx ? p.row_idx[t] : t;
        float f[C];
        lb_load_cols<C>(p.x + (size_t)src * p.ldx, k0, p.width, vec, f);
#pragma unroll
        for (int e = 0; e < C; ++e) f[e] *= s_r[tt + back];
        if (k0 < p.width) {
            float a[C], w[C], h[C];
#pragma unroll
            for (int e = 0; e < C; ++e) a[e] = 0.f;
            for (int j = 0; j < p.taps; ++j) {  // tap j looks back taps - 1 - j positions
                const int ts = t - back + j;
                if (p.pos0 + ts < 0) continue;
                lb_load_cols<C>(p.conv_w + (size_t)j * p.ring_ld, k0, p.width, vec, w);
                if (ts >= 0) {
                    lb_load_cols<C>(p.x + (size_t)ts * p.ldx, k0, p.width, vec, h);
#pragma unroll
                    for (int e = 0; e < C; ++e) h[e] *= s_r[tt + j];
                } else {
                    lb_load_cols<C>(p.ring + (size_t)((p.pos0 + ts) % p.taps) * p.ring_ld, k0, p.width, vec, h);
                }
#pragma unroll
                for (int e = 0; e < C; ++e) a[e] = fmaf(w[e], h[e], a[e]);
            }
#pragma unroll
            for (int e = 0; e < C; ++e) f[e] += a[e];
        }
        *reinterpret_cast<uint4*>(p.img + lb_img_chunk(t, c, p.slices)) = lb_pack_chunk<WT>(f);
    }
}

// the same without a convolution, a CTA per token with the row in registers as far as it fits
template <typename WT>
__global__ void __launch_bounds__(256) lb_norm_row_kernel(const LbNormBlock p, bool vec) {
    constexpr int C = LbElem<WT>::kChunk, KEEP = 32 / C;
    __shared__ float red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x, chunks = p.slices * 8;
    const float* row = p.x + (size_t)(p.row_idx ? p.row_idx[t] : t) * p.ldx;
    float f[KEEP][C], ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int c = threadIdx.x + i * 256;
        if (c < chunks) lb_load_cols<C>(row, c * C, p.width, vec, f[i]);
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if ((int)threadIdx.x + i * 256 < chunks)
#pragma unroll
            for (int e = 0; e < C; ++e) ss = fmaf(f[i][e], f[i][e], ss);
    for (int k = KEEP * 256 * C + (int)threadIdx.x; k < p.width; k += 256) ss = fmaf(row[k], row[k], ss);
    ss = lb_block_sumf(ss, red);
    const float r = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.width), p.eps))) * (p.gain ? *p.gain : 1.f);
    auto finish = [&](int c, float* g) {
#pragma unroll
        for (int e = 0; e < C; ++e) g[e] *= r;
        if (p.gain_w) {
            float w[C];
            lb_load_cols<C>(p.gain_w, c * C, p.width, vec, w);
#pragma unroll
            for (int e = 0; e < C; ++e) g[e] *= w[e];
        }
        if (p.rows) {
            float* out = p.rows + (size_t)t * p.ldx + c * C;
            if (vec && (c + 1) * C <= p.width) {
#pragma unroll
                for (int e = 0; e < C; e += 4) *reinterpret_cast<float4*>(out + e) = make_float4(g[e], g[e + 1], g[e + 2], g[e + 3]);
            } else {
#pragma unroll
                for (int e = 0; e < C; ++e)
                    if (c * C + e < p.width) out[e] = g[e];
            }
        }
        if (p.img) *reinterpret_cast<uint4*>(p.img + lb_img_chunk(t, c, p.slices)) = lb_pack_chunk<WT>(g);
    };
#pragma unroll
    for (int i = 0; i < KEEP; ++i)
        if ((int)threadIdx.x + i * 256 < chunks) finish(threadIdx.x + i * 256, f[i]);
    for (int c = threadIdx.x + KEEP * 256; c < chunks; c += 256) {
        float g[C];
        lb_load_cols<C>(row, c * C, p.width, vec, g);
        finish(c, g);
    }
}

__global__ void __launch_bounds__(256) lb_conv_commit_kernel(const LbNormBlock p) {
    __shared__ float red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = p.T - 1 - (int)blockIdx.x;
    if (t < 0) return;
    const float* row = p.x + (size_t)t * p.ldx;
    float ss = 0.f;
    for (int k = threadIdx.x; k < p.width; k += blockDim.x) ss = fmaf(row[k], row[k], ss);
    ss = lb_block_sumf(ss, red);
    const float r = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.width), p.eps))) * *p.gain;
    float* out = p.ring + (size_t)((p.pos0 + t) % p.taps) * p.ring_ld;
    for (int k = threadIdx.x; k < p.width; k += blockDim.x) out[k] = row[k] * r;
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_rows_image_kernel(const float* __restrict__ x, int ldx, int cols, int slices, uint8_t* __restrict__ img) {
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x;
    for (int c = threadIdx.x; c < slices * 8; c += blockDim.x) {
        float f[C];
        lb_load_cols<C>(x + (size_t)t * ldx, c * C, cols, ldx % 4 == 0, f);
        *reinterpret_cast<uint4*>(img + lb_img_chunk(t, c, slices)) = lb_pack_chunk<WT>(f);
    }
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_gated_heads_kernel(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg, bool vec, int heads, int vdim,
                                                             const float* __restrict__ w, bool gate_sigmoid, const float* __restrict__ scale, float eps, int slices,
                                                             uint8_t* __restrict__ img) {
    extern __shared__ float s_r[];
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, HV = heads * vdim;
    const float* row = o + (size_t)t * ldo;
    for (int h = warp; h < heads; h += 8) {
        float ss = 0.f;
        const float by = scale ? scale[(size_t)t * heads + h] : 1.f;
        for (int k = lane; k < vdim; k += 32) {
            const float v = row[(size_t)h * vdim + k] * by;
            ss = fmaf(v, v, ss);
        }
        ss = lb_warp_sumf(ss);
        if (lane == 0) s_r[h] = by * __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)vdim), eps)));
    }
    __syncthreads();
    for (int c = threadIdx.x; c < slices * 8; c += blockDim.x) {
        float f[C], g[C], hw[C];
        lb_load_cols<C>(row, c * C, HV, vec, f);
        lb_load_cols<C>(gate + (size_t)t * ldg, c * C, HV, vec, g);
        lb_load_cols<C>(w, c * C, HV, vec, hw);
#pragma unroll
        for (int e = 0; e < C; ++e) {
            const int k = c * C + e, h = k / vdim;
            f[e] = k < HV ? f[e] * s_r[h] * hw[e] * (gate_sigmoid ? lb_sigmoidf(g[e]) : lb_siluf(g[e])) : 0.f;
        }
        *reinterpret_cast<uint4*>(img + lb_img_chunk(t, c, slices)) = lb_pack_chunk<WT>(f);
    }
}

// ---- latent attention ---------------------------------------------------------------------------------------------

// what a layer with a latent projection of its own adds to the cache: rms of the projected row times a weight
struct LatentRow {
    const float* raw;  // [tokens, ldr], or null
    int ldr;
    const float* weight;
    float eps;
};

template <typename WT>
__device__ void latent_store_row(const LbLatent& p, const LatentRow& l, int t) {
    constexpr int C = LbElem<WT>::kChunk;
    __shared__ float red[8];
    const int pos = p.pos ? p.pos[t] : p.pos0 + t, lane = p.pos ? p.lane0 + t : p.lane0;
    if (pos >= p.max_seq) return;
    const float* row = l.raw + (size_t)t * l.ldr;
    float ss = 0.f;
    for (int k = threadIdx.x; k < p.rank; k += blockDim.x) ss = fmaf(row[k], row[k], ss);
    ss = lb_block_sumf(ss, red);
    const float r = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.rank), l.eps)));
    uint8_t* img = p.cache + (size_t)lane * p.lane_bytes;
    for (int c = threadIdx.x; c < p.slices * 8; c += blockDim.x) {
        float f[C];
#pragma unroll
        for (int e = 0; e < C; ++e) f[e] = c * C + e < p.rank ? row[c * C + e] * r * l.weight[c * C + e] : 0.f;
        *reinterpret_cast<uint4*>(img + lb_img_chunk(pos, c, p.slices)) = lb_pack_chunk<WT>(f);
    }
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_latent_store_kernel(const LbLatent p, const LatentRow l) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    latent_store_row<WT>(p, l, blockIdx.x);
}

// CTA = (32 chunks of the latent, head, token): thread = (row % 8, chunk), the rows of the head in groups of eight.  One CTA more
// per token puts the token's latent into the cache.
template <typename WT>
__global__ void __launch_bounds__(256) lb_absorb_q_kernel(const LbLatent p, const LatentRow l, float* __restrict__ ql) {
    extern __shared__ float sm[];
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.y, t = blockIdx.z;
    if (h == p.heads) {
        if (blockIdx.x == 0) latent_store_row<WT>(p, l, t);
        return;
    }
    const int r8 = threadIdx.x & 7, chunk = blockIdx.x * 32 + (threadIdx.x >> 3);
    float* sq = sm;  // [dim]
    for (int d = threadIdx.x; d < p.dim; d += blockDim.x) sq[d] = p.q[(size_t)t * p.ldq + h * p.dim + d] * p.scale;
    __syncthreads();
    float acc[C];
#pragma unroll
    for (int e = 0; e < C; ++e) acc[e] = 0.f;
    if (chunk < p.slices * 8) {
#pragma unroll 4
        for (int d = r8; d < p.dim; d += 8) {
            float f[C];
            lb_unpack_chunk<WT>(__ldg(reinterpret_cast<const uint4*>(p.uk + lb_img_chunk(h * p.dim + d, chunk, p.slices))), f);
#pragma unroll
            for (int e = 0; e < C; ++e) acc[e] = fmaf(sq[d], f[e], acc[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < C; ++e) {
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 1);
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 2);
        acc[e] += __shfl_xor_sync(0xffffffffu, acc[e], 4);
    }
    if (r8 == 0 && chunk < p.slices * 8) {
        float* out = ql + ((size_t)t * p.heads + h) * p.rank;
#pragma unroll
        for (int e = 0; e < C; ++e)
            if (chunk * C + e < p.rank) out[chunk * C + e] = acc[e];
    }
}

// CTA = (32 value rows, head, token): a warp per row
template <typename WT>
__global__ void __launch_bounds__(256) lb_absorb_v_kernel(const LbLatent p, const float* __restrict__ ol, float* __restrict__ out, int ldo) {
    extern __shared__ float sm[];
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.y, t = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float* row = ol + ((size_t)t * p.heads + h) * p.rank;
    for (int k = threadIdx.x; k < p.slices * 8 * C; k += blockDim.x) sm[k] = k < p.rank ? row[k] : 0.f;
    __syncthreads();
    for (int i = warp; i < 32; i += 8) {
        const int v = blockIdx.x * 32 + i;
        if (v >= p.vdim) break;
        float a = 0.f;
        for (int c = lane; c < p.slices * 8; c += 32) {
            float f[C];
            lb_unpack_chunk<WT>(__ldg(reinterpret_cast<const uint4*>(p.uv + lb_img_chunk(h * p.vdim + v, c, p.slices))), f);
#pragma unroll
            for (int e = 0; e < C; ++e) a = fmaf(f[e], sm[c * C + e], a);
        }
        a = lb_warp_sumf(a);
        if (lane == 0) out[(size_t)t * ldo + h * p.vdim + v] = a;
    }
}

// One CTA per (head, token), any precision: tiles of 256 positions, a thread per position for the scores, then a thread per
// (latent chunk, position group) for the weighted sum; running maximum and sum over the tiles.
constexpr int kLatTile = 256;
template <typename WT>
__global__ void __launch_bounds__(256) lb_latent_attn_kernel(const LbLatent p, const float* __restrict__ ql, float* __restrict__ ol, int PG) {
    extern __shared__ __align__(16) float sm[];
    constexpr int C = LbElem<WT>::kChunk;
    __shared__ float sw[kLatTile], red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, chunks = p.slices * 8;
    const int pos = p.pos ? p.pos[t] : p.pos0 + t, seq = p.pos ? p.lane0 + t : p.lane0;
    const uint8_t* img = p.cache + (size_t)seq * p.lane_bytes;
    float* sq = sm;                 // [chunks * C]
    float* so = sm + chunks * C;    // [chunks * C] (times PG for the final sum)
    for (int k = tid; k < chunks * C; k += 256) sq[k] = k < p.rank ? ql[((size_t)t * p.heads + h) * p.rank + k] : 0.f;
    const int pg = tid % PG, c0 = tid / PG;
    float acc[C];
#pragma unroll
    for (int e = 0; e < C; ++e) acc[e] = 0.f;
    float mx = -INFINITY, den = 0.f;
    __syncthreads();
    for (int j0 = 0; j0 <= pos; j0 += kLatTile) {
        const int j = j0 + tid;
        float sc = -INFINITY;
        if (j <= pos) {
            sc = 0.f;
#pragma unroll 4
            for (int c = 0; c < chunks; ++c) {
                float f[C];
                lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(img + lb_img_chunk(j, c, p.slices)), f);
#pragma unroll
                for (int e = 0; e < C; ++e) sc = fmaf(f[e], sq[c * C + e], sc);
            }
        }
        float m = sc;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        if ((tid & 31) == 0) red[tid >> 5] = m;
        __syncthreads();
        for (int i = 0; i < 8; ++i) m = fmaxf(m, red[i]);
        const float nm = fmaxf(mx, m), f = expf(mx - nm), w = j <= pos ? expf(sc - nm) : 0.f;
        mx = nm;
        sw[tid] = w;
        den = den * f + lb_block_sumf(w, red);  // (its barriers also publish sw)
        if (c0 < chunks) {
#pragma unroll
            for (int e = 0; e < C; ++e) acc[e] *= f;
            const int n = min(kLatTile, pos + 1 - j0);
#pragma unroll 4
            for (int i = pg; i < n; i += PG) {
                float c[C];
                lb_unpack_chunk<WT>(*reinterpret_cast<const uint4*>(img + lb_img_chunk(j0 + i, c0, p.slices)), c);
#pragma unroll
                for (int e = 0; e < C; ++e) acc[e] = fmaf(sw[i], c[e], acc[e]);
            }
        }
        __syncthreads();
    }
    if (c0 < chunks) {
#pragma unroll
        for (int e = 0; e < C; ++e) so[((size_t)pg * chunks + c0) * C + e] = acc[e];
    }
    __syncthreads();
    for (int k = tid; k < p.rank; k += 256) {
        float o = 0.f;
        for (int g = 0; g < PG; ++g) o += so[(size_t)g * chunks * C + k];
        ol[((size_t)t * p.heads + h) * p.rank + k] = __fdiv_rn(o, den);
    }
}

// ---- routing ----------------------------------------------------------------------------------------------------

__global__ void __launch_bounds__(256) lb_route_topk_kernel(const LbRouteBlock p) {
    extern __shared__ float sm[];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x * 8 + warp;
    if (t >= p.T) return;
    float* row = sm + (size_t)warp * p.experts;
    for (int e = lane; e < p.experts; e += 32) row[e] = p.logits[(size_t)t * p.ldl + e];
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
            row[bi] = -INFINITY;
            p.idx[(size_t)t * p.top + j] = bi;
            p.score[(size_t)t * p.top + j] = lb_sigmoidf(p.logits[(size_t)t * p.ldl + bi]);
            p.slot[(size_t)t * p.top + j] = atomicAdd(p.count + bi, 1);  // the order inside an expert does not matter: its rows are independent
        }
        __syncwarp();
    }
}

__global__ void __launch_bounds__(256) lb_route_plan_kernel(const LbRouteBlock p) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    if (threadIdx.x == 0) {
        int b = 0;
        for (int e = 0; e < p.experts; ++e) {
            p.offset[e] = b * kImgRows;
            const int n = lb_ceil_div(p.count[e], kImgRows);
            for (int i = 0; i < n; ++i) p.block_group[b + i] = e;
            b += n;
            p.count[e] = 0;  // zero between launches
        }
        *p.nblocks = b;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < p.T * p.top; i += blockDim.x) p.slot[i] += p.offset[p.idx[i]];
}

template <typename WT>
__global__ void __launch_bounds__(256) lb_route_gather_kernel(const LbRouteBlock p, const float* __restrict__ x, int ldx, int width, const float* gain,
                                                              float eps, int slices, uint8_t* __restrict__ img) {
    constexpr int C = LbElem<WT>::kChunk;
    __shared__ float red[8];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x;
    const float* row = x + (size_t)t * ldx;
    float ss = 0.f;
    for (int k = threadIdx.x; k < width; k += blockDim.x) ss = fmaf(row[k], row[k], ss);
    ss = lb_block_sumf(ss, red);
    const float r = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)width), eps))) * *gain;
    for (int c = threadIdx.x; c < slices * 8; c += blockDim.x) {
        float h[C];
        lb_load_cols<C>(row, c * C, width, ldx % 4 == 0, h);
#pragma unroll
        for (int e = 0; e < C; ++e) h[e] *= r;
        for (int j = 0; j < p.top; ++j) {
            const float w = p.score[(size_t)t * p.top + j];
            float f[C];
#pragma unroll
            for (int e = 0; e < C; ++e) f[e] = w * h[e];
            *reinterpret_cast<uint4*>(img + lb_img_chunk(p.slot[(size_t)t * p.top + j], c, slices)) = lb_pack_chunk<WT>(f);
        }
    }
}

__global__ void __launch_bounds__(256) lb_route_combine_kernel(const LbRouteBlock p, const float* __restrict__ y, int ldy, float mult, int width,
                                                               float* __restrict__ x, int ldx) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x;
    for (int k = threadIdx.x; k < width; k += blockDim.x) {
        float a = 0.f;
        for (int j = 0; j < p.top; ++j) a += y[(size_t)p.slot[(size_t)t * p.top + j] * ldy + k];
        float* o = x + (size_t)t * ldx + k;
        *o = fmaf(mult, a, *o);
    }
}

bool bf16(int dtype) { return dtype == LOOM_B200_DTYPE_BF16; }
#define LB_TYPED(dtype, kern_f, kern_b, grid, block, smem, ...)         \
    do {                                                                \
        if (bf16(dtype))                                                \
            LB_LAUNCH(ctx, kern_b, grid, block, smem, __VA_ARGS__);     \
        else                                                            \
            LB_LAUNCH(ctx, kern_f, grid, block, smem, __VA_ARGS__);     \
    } while (0)

}  // namespace

int lb_embed_norm(loom_b200_ctx* ctx, int dtype, const void* table, int vocab, int width, const int* tok, int n, const float* gain, float eps,
                  float* x, int ldx) {
    if (bf16(dtype))
        LB_LAUNCH(ctx, lb_embed_norm_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, static_cast<const __nv_bfloat16*>(table), vocab, width, tok, gain, eps, x, ldx);
    else
        LB_LAUNCH(ctx, lb_embed_norm_kernel<float>, dim3(n), dim3(256), 0, static_cast<const float*>(table), vocab, width, tok, gain, eps, x, ldx);
    return 0;
}

int lb_embed_image(loom_b200_ctx* ctx, int dtype, const uint8_t* img, int slices, int vocab, int width, const int* tok, int n, float* x, int ldx) {
    LB_TYPED(dtype, lb_embed_image_kernel<float>, lb_embed_image_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, img, slices, vocab, width, tok, x, ldx);
    return 0;
}

int lb_norm_block(loom_b200_ctx* ctx, int dtype, const LbNormBlock& p) {
    LB_REQUIRE(ctx, p.taps >= 1 && p.taps <= kMaxTaps, "norm_block: %d taps (1..%d)", p.taps, kMaxTaps);
    if (!p.conv_w) {
        LB_TYPED(dtype, lb_norm_row_kernel<float>, lb_norm_row_kernel<__nv_bfloat16>, dim3(p.T), dim3(256), 0, p,
                 lb_vec_rows(p.x, p.ldx) && (!p.gain_w || lb_vec_rows(p.gain_w, 4)) && (!p.rows || lb_vec_rows(p.rows, p.ldx)));
        return 0;
    }
    LB_TYPED(dtype, lb_norm_conv_kernel<float>, lb_norm_conv_kernel<__nv_bfloat16>, dim3(lb_ceil_div(p.T, kNormTokens)), dim3(256), 0, p,
             lb_vec_rows(p.x, p.ldx) && lb_vec_rows(p.conv_w, p.ring_ld) && lb_vec_rows(p.ring, p.ring_ld));
    return 0;
}

int lb_conv_commit(loom_b200_ctx* ctx, const LbNormBlock& p) {
    if (p.taps < 2) return 0;
    LB_LAUNCH(ctx, lb_conv_commit_kernel, dim3(p.taps - 1), dim3(256), 0, p);
    return 0;
}

int lb_rows_image(loom_b200_ctx* ctx, int dtype, const float* x, int ldx, int T, int cols, int slices, uint8_t* img) {
    LB_TYPED(dtype, lb_rows_image_kernel<float>, lb_rows_image_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, x, ldx, cols, slices, img);
    return 0;
}

int lb_gated_heads_image(loom_b200_ctx* ctx, int dtype, const float* o, int ldo, const float* gate, int ldg, int T, int heads, int vdim, const float* head_w,
                         bool gate_sigmoid, const float* scale, float eps, int slices, uint8_t* img) {
    LB_TYPED(dtype, lb_gated_heads_kernel<float>, lb_gated_heads_kernel<__nv_bfloat16>, dim3(T), dim3(256), (size_t)heads * sizeof(float), o, ldo, gate, ldg,
             lb_vec_rows(o, ldo) && lb_vec_rows(gate, ldg) && lb_vec_rows(head_w, 4), heads, vdim, head_w, gate_sigmoid, scale, eps, slices, img);
    return 0;
}

int lb_latent_store(loom_b200_ctx* ctx, int dtype, const LbLatent& p, const float* raw, int ldr, const float* weight, float eps, int tokens) {
    const LatentRow l = {raw, ldr, weight, eps};
    LB_TYPED(dtype, lb_latent_store_kernel<float>, lb_latent_store_kernel<__nv_bfloat16>, dim3(tokens), dim3(256), 0, p, l);
    return 0;
}

int lb_latent_absorb_q(loom_b200_ctx* ctx, int dtype, const LbLatent& p, const float* raw, int ldr, const float* weight, float eps, int tokens, float* ql) {
    LB_REQUIRE(ctx, p.dim <= 8192, "latent attention: query dimension %d", p.dim);
    const LatentRow l = {raw, ldr, weight, eps};
    LB_TYPED(dtype, lb_absorb_q_kernel<float>, lb_absorb_q_kernel<__nv_bfloat16>, dim3(lb_ceil_div(p.slices * 8, 32), p.heads + (raw ? 1 : 0), tokens), dim3(256),
             (size_t)p.dim * sizeof(float), p, l, ql);
    return 0;
}

int lb_latent_absorb_v(loom_b200_ctx* ctx, int dtype, const LbLatent& p, int tokens, const float* ol, float* out, int ldo) {
    const size_t smem = (size_t)p.slices * lb_slice_cols(dtype) * sizeof(float);
    LB_REQUIRE(ctx, smem <= 48 * 1024, "latent attention: latent size %d", p.rank);
    LB_TYPED(dtype, lb_absorb_v_kernel<float>, lb_absorb_v_kernel<__nv_bfloat16>, dim3(lb_ceil_div(p.vdim, 32), p.heads, tokens), dim3(256), smem, p, ol, out, ldo);
    return 0;
}

int lb_latent_attention(loom_b200_ctx* ctx, int dtype, const LbLatent& p, int tokens, const float* ql, float* ol) {
    const int chunks = p.slices * 8;
    LB_REQUIRE(ctx, chunks <= 256, "latent attention: latent size %d", p.rank);
    int PG = 1;
    while (PG * 2 * chunks <= 256) PG *= 2;
    const size_t smem = (size_t)chunks * (16 / (bf16(dtype) ? 2 : 4)) * (1 + PG) * sizeof(float);
    LB_TYPED(dtype, lb_latent_attn_kernel<float>, lb_latent_attn_kernel<__nv_bfloat16>, dim3(p.heads, tokens), dim3(256), smem, p, ql, ol, PG);
    return 0;
}

int lb_route_block(loom_b200_ctx* ctx, const LbRouteBlock& p) {
    const size_t smem = (size_t)8 * p.experts * sizeof(float);
    LB_REQUIRE(ctx, smem <= 48 * 1024, "routing: %d experts", p.experts);
    LB_LAUNCH(ctx, lb_route_topk_kernel, dim3(lb_ceil_div(p.T, 8)), dim3(256), smem, p);
    LB_LAUNCH(ctx, lb_route_plan_kernel, dim3(1), dim3(256), 0, p);
    return 0;
}

int lb_route_gather(loom_b200_ctx* ctx, int dtype, const LbRouteBlock& p, const float* x, int ldx, int width, const float* gain, float eps, int slices,
                    uint8_t* img) {
    LB_TYPED(dtype, lb_route_gather_kernel<float>, lb_route_gather_kernel<__nv_bfloat16>, dim3(p.T), dim3(256), 0, p, x, ldx, width, gain, eps, slices, img);
    return 0;
}

int lb_route_combine(loom_b200_ctx* ctx, const LbRouteBlock& p, const float* y, int ldy, float mult, int width, float* x, int ldx) {
    LB_LAUNCH(ctx, lb_route_combine_kernel, dim3(p.T), dim3(256), 0, p, y, ldy, mult, width, x, ldx);
    return 0;
}
