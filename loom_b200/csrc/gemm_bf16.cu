// gemm_bf16.cu -- token-block GEMM of bf16 matrices on the 5th-generation tensor cores (tcgen05, kind::f16).
//
//   D[128 tokens, N rows] (float, TMEM) += X[128 tokens, 64] (bf16, shared) * W[N rows, 64]^T (bf16, shared)
//
// The same machine as the persistent int8 GEMM (gemm_ternary_i8.cu): both operands are stored in HBM as the shared-memory
// image the tensor core reads (dense.cuh), a load warp brings one K slice of 64 columns per pipeline stage with two or three
// bulk copies, one elected thread issues four K = 16 MMAs per slice, tensor memory holds two accumulator buffers and eight
// epilogue warps drain tile i while tile i + 1 accumulates.  Tokens are the M side, so a thread of the epilogue owns a
// token and eight consecutive output columns of it are one 16-byte chunk of the next product's input image.
// N is 256 (two row blocks, or a gate and an up block side by side) or 128.  Routed experts: the token blocks of the image
// are grouped by expert and a table names each block's expert; the number of blocks in use is read on the device.
// Every mbarrier wait is bounded; on expiry the kernel raises the context's status word, frees its tensor memory and returns.
#include "dense.cuh"
#include "umma.cuh"

namespace {

constexpr int kEpiThreads = 256;
constexpr int kMmaWarp = kEpiThreads / 32, kLoadWarp = kMmaWarp + 1;
constexpr int kThreads = kEpiThreads + 64;

template <int NB>
struct Cfg {
    static constexpr int kStageBytes = kImgBlock * (1 + NB);
    static constexpr int kStages = (200 * 1024) / kStageBytes > 6 ? 6 : (200 * 1024) / kStageBytes;
    static constexpr int kCols = 128 * NB;  // TMEM columns of one accumulator buffer
    static constexpr size_t kSmem = (size_t)kStages * kStageBytes + 1024;
};

// NB = 128-row blocks of W side by side in one tile (GLU: block 0 of the gate, block 1 of the up matrix)
template <int NB, int EPI>
__global__ void __launch_bounds__(kThreads, 1) lb_gemm_bf16_kernel(const LbDenseGemm p, int row_tiles) {
    using C = Cfg<NB>;
    constexpr bool kDual = EPI == LB_DEPI_GLU || EPI == LB_DEPI_SILU;
    extern __shared__ __align__(1024) uint8_t smem[];
    __shared__ __align__(8) uint64_t load_bar[C::kStages], empty_bar[C::kStages], acc_full[2], acc_empty[2];
    __shared__ uint32_t tmem_base_s;
    __shared__ int s_failed;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nrb = lb_ceil_div(p.rows, kImgRows);  // 128-row blocks of W

    if (tid == 0) {
        for (int s = 0; s < C::kStages; ++s) {
            lb_mbar_init(&load_bar[s], 1);
            lb_mbar_init(&empty_bar[s], 1);
        }
        for (int b = 0; b < 2; ++b) {
            lb_mbar_init(&acc_full[b], 1);
            lb_mbar_init(&acc_empty[b], kEpiThreads / 32);
        }
        lb_fence_mbar_init();
        s_failed = 0;
    }
    if (warp == kMmaWarp) lb_tmem_alloc(&tmem_base_s, 2 * C::kCols);
    lb_tc_fence_before();
    __syncthreads();
    lb_tc_fence_after();
    const uint32_t tmem_base = tmem_base_s;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int nblocks = p.nblocks ? *p.nblocks : lb_ceil_div(p.tokens, kImgRows);
    const int ntiles = nblocks * row_tiles;
    const int my_tiles = (int)blockIdx.x < ntiles ? (ntiles - (int)blockIdx.x + (int)gridDim.x - 1) / (int)gridDim.x : 0;

    if (warp == kLoadWarp) {
        bool failed = false;
        uint32_t it = 0;
        for (int i = 0; i < my_tiles && !failed; ++i) {
            const int t = (int)blockIdx.x + i * (int)gridDim.x;
            const int rt = t % row_tiles, tb = t / row_tiles;
            const uint8_t* xb = p.x + (size_t)tb * p.slices * kImgBlock;
            const size_t goff = p.block_group ? (size_t)p.block_group[tb] * p.group_bytes : 0;
            const uint8_t* wb[2];
            int nw = NB;
            if (kDual) {
                wb[0] = p.w + goff + (size_t)rt * p.slices * kImgBlock;
                wb[1] = p.w2 + goff + (size_t)rt * p.slices * kImgBlock;
            } else {
                wb[0] = p.w + goff + (size_t)(rt * NB) * p.slices * kImgBlock;
                wb[1] = wb[0] + (size_t)p.slices * kImgBlock;
                if (NB == 2 && rt * NB + 1 >= nrb) nw = 1;  // the second half of the last tile has no rows: its columns are never read
            }
            for (int ks = 0; ks < p.slices; ++ks, ++it) {
                const int s = (int)(it % C::kStages);
                if (it >= (uint32_t)C::kStages && !lb_mbar_wait_bounded(&empty_bar[s], (it / C::kStages - 1) & 1, kTcWaitLimit)) {
                    failed = true;
                    break;
                }
                if (lane == 0) {
                    uint8_t* st = smem + (size_t)s * C::kStageBytes;
                    lb_mbar_expect_tx(&load_bar[s], (uint32_t)(kImgBlock * (1 + nw)));
                    lb_bulk_g2s(st, xb + (size_t)ks * kImgBlock, kImgBlock, &load_bar[s]);
                    lb_bulk_g2s(st + kImgBlock, wb[0] + (size_t)ks * kImgBlock, kImgBlock, &load_bar[s]);
                    if (nw == 2) lb_bulk_g2s(st + 2 * kImgBlock, wb[1] + (size_t)ks * kImgBlock, kImgBlock, &load_bar[s]);
                }
                __syncwarp();
            }
        }
        if (failed && lane == 0) atomicExch(&s_failed, 1);
    } else if (warp == kMmaWarp) {
        constexpr uint32_t idesc = lb_idesc_bf16(128, 128 * NB, false);
        bool failed = false;
        uint32_t it = 0;
        for (int i = 0; i < my_tiles && !failed; ++i) {
            const int buf = i & 1;
            if (i >= 2 && !lb_mbar_wait_bounded(&acc_empty[buf], (uint32_t)(((i >> 1) - 1) & 1), kTcWaitLimit)) {
                failed = true;
                break;
            }
            lb_tc_fence_after();
            const uint32_t d = tmem_base + (uint32_t)(buf * C::kCols);
            for (int ks = 0; ks < p.slices; ++ks, ++it) {
                const int s = (int)(it % C::kStages);
                if (!lb_mbar_wait_bounded(&load_bar[s], (it / C::kStages) & 1, kTcWaitLimit)) {
                    failed = true;
                    break;
                }
                lb_tc_fence_after();
                if (lane == 0) {
                    const uint32_t a = lb_smem_u32(smem + (size_t)s * C::kStageBytes), b = a + kImgBlock;
#pragma unroll
                    for (int k = 0; k < 4; ++k) lb_mma_f16(d, lb_smem_desc(a + k * 256, 128, 1024), lb_smem_desc(b + k * 256, 128, 1024), idesc, (ks > 0 || k > 0) ? 1u : 0u);
                    lb_mma_commit(&empty_bar[s]);
                }
                __syncwarp();
            }
            if (!failed && lane == 0) lb_mma_commit(&acc_full[buf]);
            __syncwarp();
        }
        if (failed && lane == 0) atomicExch(&s_failed, 1);
        lb_tc_fence_before();
    } else {
        // a warp reads the 32 TMEM lanes (= tokens) of its quarter; the two warps of a quarter split the columns
        const int quarter = warp & 3, half = warp >> 2;
        constexpr int kOut = kDual ? 128 : 128 * NB;  // output columns of a tile
        bool failed = false;
        for (int i = 0; i < my_tiles && !failed; ++i) {
            const int t = (int)blockIdx.x + i * (int)gridDim.x;
            const int rt = t % row_tiles, tb = t / row_tiles, buf = i & 1;
            if (!lb_mbar_wait_bounded(&acc_full[buf], (uint32_t)((i >> 1) & 1), kTcWaitLimit)) {
                failed = true;
                if (lane == 0) atomicExch(&s_failed, 1);
                break;
            }
            lb_tc_fence_after();
            const int tok = tb * kImgRows + quarter * 32 + lane;
            const bool tok_ok = p.nblocks || tok < p.tokens;
            const uint32_t tacc = tmem_base + (uint32_t)(buf * C::kCols) + ((uint32_t)(quarter * 32) << 16);
#pragma unroll 1
            for (int c0 = half * (kOut / 2); c0 < (half + 1) * (kOut / 2); c0 += 16) {
                float v[16], u[16];
                lb_tmem_ld16(tacc + (uint32_t)c0, v);
                if (kDual) lb_tmem_ld16(tacc + (uint32_t)(128 + c0), u);
                lb_tmem_wait_ld();
#pragma unroll
                for (int hh = 0; hh < 2; ++hh) {
                    const int r = rt * kOut + c0 + 8 * hh;
                    const float *v8 = v + 8 * hh, *u8 = u + 8 * hh;
                    if (!tok_ok) continue;
                    if (EPI == LB_DEPI_F32 || EPI == LB_DEPI_RESID) {
                        if (r >= p.ldo) continue;
                        float4* o = reinterpret_cast<float4*>(p.out + (size_t)tok * p.ldo + r);
                        if (EPI == LB_DEPI_F32) {
                            o[0] = make_float4(v8[0], v8[1], v8[2], v8[3]);
                            o[1] = make_float4(v8[4], v8[5], v8[6], v8[7]);
                        } else {
                            float4 x = o[0], y = o[1];
                            x.x = fmaf(p.mult, v8[0], p.res_mult * x.x);
                            x.y = fmaf(p.mult, v8[1], p.res_mult * x.y);
                            x.z = fmaf(p.mult, v8[2], p.res_mult * x.z);
                            x.w = fmaf(p.mult, v8[3], p.res_mult * x.w);
                            y.x = fmaf(p.mult, v8[4], p.res_mult * y.x);
                            y.y = fmaf(p.mult, v8[5], p.res_mult * y.y);
                            y.z = fmaf(p.mult, v8[6], p.res_mult * y.z);
                            y.w = fmaf(p.mult, v8[7], p.res_mult * y.w);
                            o[0] = x;
                            o[1] = y;
                        }
                    } else {
                        if (EPI == LB_DEPI_HEADS ? r >= p.rows : r / 64 >= p.img_slices) continue;
                        float f[8];
#pragma unroll
                        for (int j = 0; j < 8; ++j) {
                            f[j] = v8[j];
                            if (EPI == LB_DEPI_GELU) f[j] = lb_gelu_erff(v8[j]);
                            if (EPI == LB_DEPI_GLU) f[j] = lb_clamped_glu(v8[j], u8[j], p.limit);
                            if (EPI == LB_DEPI_SILU) f[j] = lb_siluf(v8[j]) * u8[j];
                        }
                        if (EPI == LB_DEPI_HEADS)
                            *reinterpret_cast<uint4*>(p.img + lb_heads_chunk(tok, r, p.heads, p.head_dim, p.head_chunks)) = lb_pack_chunk<__nv_bfloat16>(f);
                        else
                            lb_img_store8<__nv_bfloat16>(p.img, tok, r, p.img_slices, f);
                    }
                }
            }
            lb_tc_fence_before();
            __syncwarp();
            if (lane == 0) lb_mbar_arrive(&acc_empty[buf]);
        }
    }
    __syncthreads();
    if (warp == kMmaWarp) {
        lb_tc_fence_after();
        lb_tmem_dealloc(tmem_base, 2 * C::kCols);
    }
    if (tid == 0 && s_failed) atomicExch(p.status, 3);
}

template <int NB, int EPI>
int launch(loom_b200_ctx* ctx, const LbDenseGemm& p) {
    using C = Cfg<NB>;
    const int per = EPI == LB_DEPI_GLU || EPI == LB_DEPI_SILU ? 1 : NB;
    const int row_tiles = lb_ceil_div(lb_ceil_div(p.rows, kImgRows), per);
    const int blocks = p.nblocks ? p.max_blocks : lb_ceil_div(p.tokens, kImgRows);
    const int ntiles = row_tiles * blocks;
    LB_BIG_SMEM(ctx, (lb_gemm_bf16_kernel<NB, EPI>), C::kSmem);
    LB_LAUNCH(ctx, (lb_gemm_bf16_kernel<NB, EPI>), dim3(ntiles < ctx->sm_count ? ntiles : ctx->sm_count), dim3(kThreads), C::kSmem, p, row_tiles);
    return 0;
}

template <int EPI>
int launch_plain(loom_b200_ctx* ctx, const LbDenseGemm& p) {
    // a tile's time follows the bytes of its stages (48 KB for two row blocks, 32 KB for one), the launch's the busiest CTA
    const int nrb = lb_ceil_div(p.rows, kImgRows), blocks = p.nblocks ? p.max_blocks : lb_ceil_div(p.tokens, kImgRows), sms = ctx->sm_count;
    const int t1 = nrb * blocks, t2 = lb_ceil_div(nrb, 2) * blocks;
    const bool wide = nrb > 1 && 3 * lb_ceil_div(t2, sms) <= 2 * lb_ceil_div(t1, sms);
    return wide ? launch<2, EPI>(ctx, p) : launch<1, EPI>(ctx, p);
}

}  // namespace

int lb_gemm_bf16_run(loom_b200_ctx* ctx, int epi, const LbDenseGemm& p) {
    switch (epi) {
        case LB_DEPI_F32: return launch_plain<LB_DEPI_F32>(ctx, p);
        case LB_DEPI_RESID: return launch_plain<LB_DEPI_RESID>(ctx, p);
        case LB_DEPI_GELU: return launch_plain<LB_DEPI_GELU>(ctx, p);
        case LB_DEPI_IMG: return launch_plain<LB_DEPI_IMG>(ctx, p);
        case LB_DEPI_HEADS: return launch_plain<LB_DEPI_HEADS>(ctx, p);
        case LB_DEPI_GLU: return launch<2, LB_DEPI_GLU>(ctx, p);
        case LB_DEPI_SILU: return launch<2, LB_DEPI_SILU>(ctx, p);
    }
    return lb_fail(ctx, LOOM_B200_ERR_UNSUPPORTED, "gemm_bf16: epilogue %d is not built", epi);
}
