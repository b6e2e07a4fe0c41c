// latent_attention.cu -- attention over cached latents in bf16: a split kernel for single tokens that reads every latent once for
// up to sixteen heads; token blocks expand per-head keys and values from the latents for the tensor-core kernel (attention_block.cu).
#include "mixers.cuh"

#include <cmath>

namespace {

__device__ __forceinline__ void mma_bf16(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t* r, const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(lb_smem_u32(p)));
}
// value = hi + lo, both bf16: the pair carries sixteen bits of the float
__device__ __forceinline__ void split_bf16(const float* f, uint4& hi, uint4& lo) {
    float h[8], l[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        h[i] = __bfloat162float(__float2bfloat16_rn(f[i]));
        l[i] = f[i] - h[i];
    }
    hi = lb_pack_chunk<__nv_bfloat16>(h);
    lo = lb_pack_chunk<__nv_bfloat16>(l);
}

// ---- one token per sequence (or a few tokens of one) ------------------------------------------------------------
//
// CTA = (position split, sixteen heads, token).  Tiles of 64 latents come as bulk copies of the cache image; eight warps take
// eight positions each for the scores (queries as bf16 pairs, so the score keeps the query's precision) and an eighth of the
// latent's chunks each for the weighted sum (weights as bf16 pairs, latents transposed by ldmatrix).
constexpr int kStTile = 64;
constexpr int kStThreads = 256;

struct StepSmem {
    size_t q, s, p, f, tile, bytes;
    int stages;
};
__host__ __device__ inline StepSmem step_smem(int chunks, int stages) {
    StepSmem m;
    m.tile = 0;
    m.q = m.tile + (size_t)stages * chunks * 1024;    // [stage][slice][8 groups][8 chunks][8][16 B]
    m.p = m.q + (size_t)2 * chunks * 256;             // queries hi / lo: [chunk][16 heads] 16 B
    m.s = m.p + 2 * 8 * 256;                          // weights hi / lo: [position chunk][16 heads] 16 B
    m.f = m.s + 16 * (kStTile + 4) * sizeof(float);   // scores
    m.bytes = m.f + 3 * 16 * sizeof(float);           // maximum, sum, rescale of every head
    m.stages = stages;
    return m;
}

template <int CPW>  // latent chunks of a warp, at most
__global__ void __launch_bounds__(kStThreads) lb_latent_step_kernel(const LbLatent p, const float* __restrict__ ql, float* __restrict__ part, int splits,
                                                                    int stages, int* status) {
    extern __shared__ __align__(128) uint8_t sm[];
    __shared__ __align__(8) uint64_t bars[2];
    const int chunks = p.slices * 8;
    const StepSmem at = step_smem(chunks, stages);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int h0 = blockIdx.y * 16, m = blockIdx.z, split = blockIdx.x;
    uint4* qs = reinterpret_cast<uint4*>(sm + at.q);
    uint4* ps = reinterpret_cast<uint4*>(sm + at.p);
    float* ss = reinterpret_cast<float*>(sm + at.s);
    float *smax = reinterpret_cast<float*>(sm + at.f), *ssum = smax + 16, *sfac = ssum + 16;
    if (tid == 0) {
        lb_mbar_init(&bars[0], 1);
        lb_mbar_init(&bars[1], 1);
        lb_fence_mbar_init();
    }
    if (tid < 16) {
        smax[tid] = -INFINITY;
        ssum[tid] = 0.f;
    }
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int pos = p.pos ? p.pos[m] : p.pos0 + m, seq = p.pos ? p.lane0 + m : p.lane0;
    const uint8_t* img = p.cache + (size_t)seq * p.lane_bytes;
    // this split's tiles: contiguous, every split within one tile of the others
    const int ntiles = pos / kStTile + 1;
    const int j0 = (int)((long long)ntiles * split / splits), j1 = (int)((long long)ntiles * (split + 1) / splits);
    __syncthreads();
    auto fetch = [&](int j) {  // a tile = half of a 128-position block: 8 KB per slice
        const int s = (j - j0) % stages;
        uint8_t* dst = sm + at.tile + (size_t)s * chunks * 1024;
        lb_mbar_expect_tx(&bars[s], (uint32_t)chunks * 1024);
        const uint8_t* src = img + (size_t)(j >> 1) * p.slices * kImgBlock + (size_t)(j & 1) * 8192;
        for (int sl = 0; sl < p.slices; ++sl) lb_bulk_g2s(dst + (size_t)sl * 8192, src + (size_t)sl * kImgBlock, 8192, &bars[s]);
    };
    if (tid == 0)
        for (int j = j0; j < j1 && j < j0 + stages; ++j) fetch(j);
    if (j0 < j1) {
        for (int i = tid; i < chunks * 16; i += kStThreads) {
            const int c = i >> 4, hh = i & 15;
            float f[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const int k = c * 8 + e;
                f[e] = h0 + hh < p.heads && k < p.rank ? ql[((size_t)m * p.heads + h0 + hh) * p.rank + k] : 0.f;
            }
            split_bf16(f, qs[i], qs[chunks * 16 + i]);
        }
    }
    __syncthreads();
    float o[CPW][4];
#pragma unroll
    for (int i = 0; i < CPW; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    const int cw = lb_ceil_div(chunks, 8), c0 = warp * cw, c1 = min(chunks, c0 + cw);
    bool failed = false;
    for (int j = j0; j < j1; ++j) {
        const int s = (j - j0) % stages;
        if (!failed && !lb_mbar_wait_bounded(&bars[s], (uint32_t)(((j - j0) / stages) & 1))) {
            failed = true;
            if (lane == 0) atomicExch(status, 1);
        }
        const uint8_t* tile = sm + at.tile + (size_t)s * chunks * 1024;
        // scores of positions j*64 + warp*8 + 0..7
        float d[4] = {0.f, 0.f, 0.f, 0.f};
        for (int c = 0; c < chunks; c += 4) {
            const int ct = c + t;
            const uint4 b = *reinterpret_cast<const uint4*>(tile + (size_t)(ct >> 3) * 8192 + warp * 1024 + (ct & 7) * 128 + g * 16);
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const uint4 a0 = qs[half * chunks * 16 + ct * 16 + g], a1 = qs[half * chunks * 16 + ct * 16 + g + 8];
                mma_bf16(d, a0.x, a1.x, a0.y, a1.y, b.x, b.y);
                mma_bf16(d, a0.z, a1.z, a0.w, a1.w, b.z, b.w);
            }
        }
        {
            const int n = warp * 8 + 2 * t, key = j * kStTile + n;
            ss[g * (kStTile + 4) + n] = key <= pos ? d[0] : -INFINITY;
            ss[g * (kStTile + 4) + n + 1] = key + 1 <= pos ? d[1] : -INFINITY;
            ss[(g + 8) * (kStTile + 4) + n] = key <= pos ? d[2] : -INFINITY;
            ss[(g + 8) * (kStTile + 4) + n + 1] = key + 1 <= pos ? d[3] : -INFINITY;
        }
        __syncthreads();
        // softmax of the tile: sixteen threads per head, four positions each (every tile has a visible position)
        {
            const int hh = tid >> 4, q = tid & 15;
            const float4 x = *reinterpret_cast<const float4*>(ss + hh * (kStTile + 4) + q * 4);
            float mx = fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w));
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
            const float old = smax[hh], nm = fmaxf(old, mx);
            float w[4] = {expf(x.x - nm), expf(x.y - nm), expf(x.z - nm), expf(x.w - nm)};
            float sum = (w[0] + w[1]) + (w[2] + w[3]);
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            __syncwarp();
            if (q == 0) {
                const float f = expf(old - nm);
                smax[hh] = nm;
                sfac[hh] = f;
                ssum[hh] = fmaf(ssum[hh], f, sum);
            }
            float l[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const float hi = __bfloat162float(__float2bfloat16_rn(w[e]));
                l[e] = w[e] - hi;
                w[e] = hi;
            }
            uint2* dst = reinterpret_cast<uint2*>(ps + (q >> 1) * 16 + hh) + (q & 1);
            *dst = make_uint2(lb_pack_bf16(w[0], w[1]), lb_pack_bf16(w[2], w[3]));
            *(dst + 2 * 8 * 16) = make_uint2(lb_pack_bf16(l[0], l[1]), lb_pack_bf16(l[2], l[3]));
        }
        __syncthreads();
        // weighted sum: A = weights [16 heads x 16 positions], B = latents transposed [16 positions x 8 columns]
        {
            const float f0 = sfac[g], f1 = sfac[g + 8];
#pragma unroll
            for (int i = 0; i < CPW; ++i) {
                o[i][0] *= f0;
                o[i][1] *= f0;
                o[i][2] *= f1;
                o[i][3] *= f1;
            }
#pragma unroll
            for (int pp = 0; pp < 2; ++pp) {  // 32 positions: two k-steps
                uint32_t a[2][2][4];          // [hi / lo][k-step]
#pragma unroll
                for (int half = 0; half < 2; ++half)
#pragma unroll
                    for (int ks = 0; ks < 2; ++ks) {
                        // positions 16 (2 pp + ks) + {2t, 2t+1} and + 8: word t of chunks 2 (2 pp + ks) and + 1
                        const uint32_t* c = reinterpret_cast<const uint32_t*>(ps + half * 128 + (2 * (2 * pp + ks)) * 16);
                        a[half][ks][0] = c[g * 4 + t];
                        a[half][ks][1] = c[(g + 8) * 4 + t];
                        a[half][ks][2] = c[64 + g * 4 + t];
                        a[half][ks][3] = c[64 + (g + 8) * 4 + t];
                    }
#pragma unroll
                for (int i = 0; i < CPW; ++i) {
                    const int c = c0 + i;
                    if (c < c1) {
                        uint32_t b[4];  // four groups of eight positions of chunk c
                        ldmatrix_x4_trans(b, tile + (size_t)(c >> 3) * 8192 + (size_t)(pp * 4 + (lane >> 3)) * 1024 + (c & 7) * 128 + (lane & 7) * 16);
#pragma unroll
                        for (int half = 0; half < 2; ++half) {
                            mma_bf16(o[i], a[half][0][0], a[half][0][1], a[half][0][2], a[half][0][3], b[0], b[1]);
                            mma_bf16(o[i], a[half][1][0], a[half][1][1], a[half][1][2], a[half][1][3], b[2], b[3]);
                        }
                    }
                }
            }
        }
        __syncthreads();  // the tile and the weights are free again
        if (tid == 0 && j + stages < j1) {
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            fetch(j + stages);
        }
    }
    // partial result: [token][head][split] {rank sums, maximum, sum}
    const int row = p.rank + 2;
#pragma unroll
    for (int hb = 0; hb < 2; ++hb) {
        const int h = h0 + g + 8 * hb;
        if (h >= p.heads) continue;
        float* out = part + (((size_t)m * p.heads + h) * splits + split) * row;
        if (j0 < j1) {
#pragma unroll
            for (int i = 0; i < CPW; ++i) {
                const int k = (c0 + i) * 8 + 2 * t;
                if (c0 + i < c1) {
                    if (k < p.rank) out[k] = o[i][2 * hb];
                    if (k + 1 < p.rank) out[k + 1] = o[i][2 * hb + 1];
                }
            }
        }
        if (warp == 0 && t == 0) {
            out[p.rank] = smax[g + 8 * hb];
            out[p.rank + 1] = ssum[g + 8 * hb];
        }
    }
}

// merges the splits, then the head's value rows: CTA = (32 value rows, head, token)
__global__ void __launch_bounds__(256) lb_latent_value_kernel(const LbLatent p, const float* __restrict__ part, int splits, float* __restrict__ out, int ldo) {
    extern __shared__ float sm2[];
    __shared__ float sw[64];
    constexpr int C = 8;
    lb_pdl_launch_dependents();
    const int h = blockIdx.y, tk = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cols = p.slices * 64, row = p.rank + 2;
    lb_pdl_wait();
    const float* base = part + ((size_t)tk * p.heads + h) * splits * row;
    if (warp == 0) {  // weight of every split: its share of the whole sum
        float mx = -INFINITY;
        for (int s = lane; s < splits; s += 32) mx = fmaxf(mx, base[(size_t)s * row + p.rank]);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        float den = 0.f;
        for (int s = lane; s < splits; s += 32) {
            const float w = expf(base[(size_t)s * row + p.rank] - mx);
            sw[s] = w;
            den = fmaf(w, base[(size_t)s * row + p.rank + 1], den);
        }
        den = lb_warp_sumf(den);
        __syncwarp();
        for (int s = lane; s < splits; s += 32) sw[s] = __fdiv_rn(sw[s], den);
    }
    __syncthreads();
    for (int k = threadIdx.x; k < cols; k += blockDim.x) {
        float a = 0.f;
        if (k < p.rank) {
            // (a split without positions has weight zero over whatever finite sums an earlier step left there)
#pragma unroll 8
            for (int s = 0; s < splits; ++s) a = fmaf(sw[s], base[(size_t)s * row + k], a);
        }
        sm2[k] = a;
    }
    __syncthreads();
    for (int i = warp; i < 32; i += 8) {
        const int v = blockIdx.x * 32 + i;
        if (v >= p.vdim) break;
        float a = 0.f;
        for (int c = lane; c < p.slices * 8; c += 32) {
            float f[C];
            lb_unpack_chunk<__nv_bfloat16>(__ldg(reinterpret_cast<const uint4*>(p.uv + lb_img_chunk(h * p.vdim + v, c, p.slices))), f);
#pragma unroll
            for (int e = 0; e < C; ++e) a = fmaf(f[e], sm2[c * C + e], a);
        }
        a = lb_warp_sumf(a);
        if (lane == 0) out[(size_t)tk * ldo + h * p.vdim + v] = a;
    }
}

// ---- token blocks: queries, expanded keys and transposed values for attention_block.cu -----------------------------------

// float query rows -> per-head bf16 blocks
__global__ void __launch_bounds__(256) lb_heads_image_kernel(const float* __restrict__ x, int ldx, int heads, int dim, int dchunks, float sign, uint8_t* __restrict__ img) {
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int t = blockIdx.x;
    for (int i = threadIdx.x; i < heads * dchunks; i += blockDim.x) {
        const int h = i / dchunks, c = i - h * dchunks;
        float f[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = c * 8 + e < dim ? sign * x[(size_t)t * ldx + h * dim + c * 8 + e] : 0.f;
        *reinterpret_cast<uint4*>(img + ((size_t)(t >> 7) * heads + h) * dchunks * 2048 + (size_t)((t & 127) >> 3) * dchunks * 128 + (size_t)c * 128 + (t & 7) * 16) =
            lb_pack_chunk<__nv_bfloat16>(f);
    }
}

template <int CPW>
int launch_step(loom_b200_ctx* ctx, const LbLatent& p, int tokens, const float* ql, float* part, int splits) {
    const int chunks = p.slices * 8;
    const int stages = step_smem(chunks, 2).bytes <= 200 * 1024 ? 2 : 1;
    const size_t smem = step_smem(chunks, stages).bytes;
    LB_BIG_SMEM(ctx, lb_latent_step_kernel<CPW>, 216 * 1024);
    LB_LAUNCH(ctx, lb_latent_step_kernel<CPW>, dim3(splits, lb_ceil_div(p.heads, 16), tokens), dim3(kStThreads), smem, p, ql, part, splits, stages, ctx->status_dev);
    return 0;
}

}  // namespace

bool lb_latent_step_supported(const LbLatent& p) {
    const int chunks = p.slices * 8;
    return chunks <= 128 && step_smem(chunks, 1).bytes <= 216 * 1024;
}

int lb_latent_step_splits(loom_b200_ctx* ctx, const LbLatent& p, int tokens) {
    int s = 2 * ctx->sm_count / (lb_ceil_div(p.heads, 16) * tokens);
    const int tiles = lb_ceil_div(p.max_seq, kStTile);
    if (s > tiles) s = tiles;
    if (s > 64) s = 64;
    return s < 1 ? 1 : s;
}

int lb_latent_step(loom_b200_ctx* ctx, const LbLatent& p, int tokens, const float* ql, float* part, int splits, float* out, int ldo) {
    const int cpw = lb_ceil_div(p.slices * 8, 8);
    if (cpw <= 2) {
        if (int rc = launch_step<2>(ctx, p, tokens, ql, part, splits)) return rc;
    } else if (cpw <= 8) {
        if (int rc = launch_step<8>(ctx, p, tokens, ql, part, splits)) return rc;
    } else if (int rc = launch_step<16>(ctx, p, tokens, ql, part, splits)) {
        return rc;
    }
    LB_LAUNCH(ctx, lb_latent_value_kernel, dim3(lb_ceil_div(p.vdim, 32), p.heads, tokens), dim3(256), (size_t)p.slices * 64 * sizeof(float), p, part, splits, out, ldo);
    return 0;
}

int lb_latent_dchunks(int dim) { return lb_round_up(lb_ceil_div(dim, 8), 2); }

bool lb_latent_block_supported(const LbLatent& p) { return p.dim % 8 == 0 && p.dim <= 256 && p.vdim % 8 == 0 && p.vdim <= 128 && p.scale != 0.f; }

size_t lb_latent_heads_bytes(const LbLatent& p, int rows) { return (size_t)lb_ceil_div(rows, 128) * p.heads * lb_latent_dchunks(p.dim) * 2048; }

int lb_latent_block(loom_b200_ctx* ctx, const LbLatent& p, int T, uint8_t* q_img, uint8_t* k_img, uint8_t* vt_img, int vt_slices, uint8_t* out, int out_slices) {
    const int ctx_rows = p.pos0 + T, dch = lb_latent_dchunks(p.dim);
    const uint8_t* cache = p.cache + (size_t)p.lane0 * p.lane_bytes;
    LB_LAUNCH(ctx, lb_heads_image_kernel, dim3(T), dim3(256), 0, p.q, p.ldq, p.heads, p.dim, dch, p.scale < 0.f ? -1.f : 1.f, q_img);
    // keys of every position, per head
    LbDenseGemm g;
    g.x = cache;
    g.tokens = ctx_rows;
    g.w = p.uk;
    g.rows = p.heads * p.dim;
    g.slices = p.slices;
    g.img = k_img;
    g.head_dim = p.dim;
    g.head_chunks = dch;
    g.heads = p.heads;
    if (int rc = lb_dense_gemm(ctx, LOOM_B200_DTYPE_BF16, LB_DEPI_HEADS, g)) return rc;
    // values transposed: the value rows are the "tokens", the positions the columns
    g = LbDenseGemm();
    g.x = p.uv;
    g.tokens = p.heads * p.vdim;
    g.w = cache;
    g.rows = ctx_rows;
    g.slices = p.slices;
    g.img = vt_img;
    g.img_slices = vt_slices;
    if (int rc = lb_dense_gemm(ctx, LOOM_B200_DTYPE_BF16, LB_DEPI_IMG, g)) return rc;
    LbAttnBlock a;
    a.q = q_img;
    a.k = k_img;
    a.vt = vt_img;
    a.heads = a.kv_heads = p.heads;
    a.dchunks = dch;
    a.vdim = a.vrows = p.vdim;
    a.vslices = vt_slices;
    a.T = T;
    a.pos0 = p.pos0;
    a.scale_log2 = fabsf(p.scale) * 1.4426950408889634f;
    a.out = out;
    a.out_slices = out_slices;
    return lb_attn_block(ctx, a);
}
