// attention_block.cu -- softmax attention of a block of tokens on the 5th-generation tensor cores (bf16 operands, float scores).
//
// CTA = (128 query tokens, head), two CTAs per SM: a query row per thread, one thread also issues the loads and the MMAs (a
// fifth warp would cost every thread a fifth of its registers).  S = Q K^T of 64 keys and O_j = P V of the same keys are both
// fresh TMEM accumulators; the running maximum, the sum and the output row live in the thread's registers, so nothing is ever
// rescaled in tensor memory.  While the threads take in O_j, the tensor core is on S_(j+1) -- and on the other CTA's tiles.
//
// The general form adds grouped heads over a ring of positions, chunks (a position sees its own chunk only: tiles in front of the
// chunk of the first row are never read), a bias by distance (a row of a table in the L1 cache while the tile is near, one number
// beyond the last bucket), a sink (the running maximum starts at its score 0, the sum at 1) and a gate per head.
#include "mixers.cuh"
#include "umma.cuh"

namespace {

// 2^x by the hardware's approximation (two units in the last place), results below 2^-126 as zero
__device__ __forceinline__ float fast_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

constexpr int kAtKeys = 64;
constexpr int kAtThreads = 128;

template <int VC, bool GEN>  // value columns, a multiple of sixteen; the general form
__global__ void __launch_bounds__(kAtThreads, 2) lb_attn_block_kernel(const LbAttnBlock p) {
    extern __shared__ __align__(1024) uint8_t sm[];
    __shared__ __align__(8) uint64_t bar_q, bar_k[2], bar_v[2], bar_s, bar_p, bar_o;
    __shared__ uint32_t tmem_base_s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nqb = lb_ceil_div(p.T, 128), qb = nqb - 1 - (int)blockIdx.y, h = blockIdx.x;  // the longest rows of every head first
    const uint32_t qbytes = (uint32_t)p.dchunks * 2048, kbytes = (uint32_t)p.dchunks * 1024, vbytes = (uint32_t)p.vrows * 128;
    constexpr uint32_t kVStage = VC * 128;
    uint8_t *sq = sm, *sk = sq + qbytes, *sv = sk + 2 * kbytes, *sp = sv + 2 * kVStage;
    constexpr uint32_t kTmem = VC + kAtKeys <= 64 ? 64 : VC + kAtKeys <= 128 ? 128 : 256;
    constexpr uint32_t id_s = lb_idesc_bf16(128, kAtKeys, false), id_o = lb_idesc_bf16(128, VC, false);
    const int last = min(p.T, qb * 128 + 128) - 1;  // last query row of the block
    const int hk = GEN ? h / (p.heads / p.kv_heads) : h, first_pos = p.pos0 + qb * 128;
    const int tile0 = GEN && p.chunk ? (first_pos - first_pos % p.chunk) / kAtKeys : 0;  // tile of the first row's first key
    const int ntiles = (p.pos0 + last) / kAtKeys + 1 - tile0;
    if (tid == 0) {
        uint64_t* one[] = {&bar_q, &bar_k[0], &bar_k[1], &bar_v[0], &bar_v[1], &bar_s, &bar_o};
        for (auto* b : one) lb_mbar_init(b, 1);
        lb_mbar_init(&bar_p, kAtThreads);
        lb_fence_mbar_init();
    }
    if (warp == 0) lb_tmem_alloc(&tmem_base_s, kTmem);
    lb_tc_fence_before();
    __syncthreads();
    lb_tc_fence_after();
    const uint32_t tmem = tmem_base_s;
    lb_pdl_launch_dependents();
    lb_pdl_wait();

    const uint32_t a_q = lb_smem_u32(sq), a_k = lb_smem_u32(sk), a_v = lb_smem_u32(sv), a_p = lb_smem_u32(sp), sbo_d = (uint32_t)p.dchunks * 128;
    auto load = [&](int j) {
        const int s = j & 1;
        const int at = GEN ? (tile0 + j) % (p.ring / kAtKeys) : j;  // tile of the cache
        lb_mbar_expect_tx(&bar_k[s], kbytes);
        lb_bulk_g2s(sk + s * kbytes, p.k + ((size_t)(at >> 1) * p.kv_heads + hk) * p.dchunks * 2048 + (size_t)(at & 1) * kbytes, kbytes, &bar_k[s]);
        lb_mbar_expect_tx(&bar_v[s], vbytes);
        for (int r = hk * p.vrows, end = r + p.vrows; r < end;) {  // the head's rows, block of 128 rows by block
            const int n = min(end, (r & ~127) + 128) - r;
            lb_bulk_g2s(sv + s * kVStage + (uint32_t)(r - hk * p.vrows) * 128, p.vt + ((size_t)(r >> 7) * p.vslices + at) * kImgBlock + (size_t)((r & 127) >> 3) * 1024,
                        (uint32_t)n * 128, &bar_v[s]);
            r += n;
        }
    };
    auto scores = [&](int j) {
        for (int k = 0; k < p.dchunks / 2; ++k)
            lb_mma_f16(tmem, lb_smem_desc(a_q + k * 256, 128, sbo_d), lb_smem_desc(a_k + (j & 1) * kbytes + k * 256, 128, sbo_d), id_s, k > 0 ? 1u : 0u);
        lb_mma_commit(&bar_s);
    };
    bool failed = false;
    if (tid == 0) {
        lb_mbar_expect_tx(&bar_q, qbytes);
        lb_bulk_g2s(sq, p.q + ((size_t)qb * p.heads + h) * qbytes, qbytes, &bar_q);
        load(0);
        if (ntiles > 1) load(1);
        failed = !lb_mbar_wait_bounded(&bar_q, 0, kTcWaitLimit) || !lb_mbar_wait_bounded(&bar_k[0], 0, kTcWaitLimit);
        if (!failed) scores(0);
    }
    __syncwarp();

    const int row = warp * 32 + lane, tok = qb * 128 + row, qpos = p.pos0 + tok;
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    float o[VC];
#pragma unroll
    for (int c = 0; c < VC; ++c) o[c] = 0.f;
    float mx = -3e38f, sum = 0.f;  // (finite: the factor may be zero, and a tile may have no visible key)
    if (GEN && p.sink) {
        mx = 0.f;
        sum = 1.f;
    }
    const float* bias = GEN && p.bias ? p.bias + (size_t)h * p.bias_ld + kBiasFront : nullptr;
    const int low = GEN && p.chunk ? qpos - qpos % p.chunk : 0;  // first visible key of this row
    uint8_t* prow = sp + (size_t)(row >> 3) * 1024 + (row & 7) * 16;
    for (int j = 0; j < ntiles; ++j) {
        if (!lb_mbar_wait_bounded(&bar_s, (uint32_t)(j & 1), kTcWaitLimit)) failed = true;
        if (__any_sync(0xffffffffu, failed)) {  // a warp leaves together; the others' waits run out
            failed = true;
            break;
        }
        lb_tc_fence_after();
        float f;
        {
            float s[kAtKeys];
#pragma unroll
            for (int c = 0; c < kAtKeys; c += 16) lb_tmem_ld16(tmem + lanes + c, s + c);
            lb_tmem_wait_ld();
            const int vis = qpos - (tile0 + j) * kAtKeys;  // keys 0..vis of the tile are visible
            if (GEN) {
                if (!bias) {
#pragma unroll
                    for (int c = 0; c < kAtKeys; ++c) s[c] *= p.scale_log2;
                } else if (vis >= kAtKeys + p.bias_len) {
                    const float far = bias[p.bias_len - 1];
#pragma unroll
                    for (int c = 0; c < kAtKeys; ++c) s[c] = fmaf(s[c], p.scale_log2, far);
                } else {  // (the row of the table goes on in front of distance 0 and behind the last one)
                    const float* row = bias + vis;
#pragma unroll
                    for (int c = 0; c < kAtKeys; ++c) s[c] = fmaf(s[c], p.scale_log2, __ldg(row - c));
                }
            }
            if (vis < kAtKeys - 1) {
#pragma unroll
                for (int c = 0; c < kAtKeys; ++c) s[c] = c <= vis ? s[c] : -INFINITY;
            }
            if (GEN && low > (tile0 + j) * kAtKeys) {
                const int from = low - (tile0 + j) * kAtKeys;
#pragma unroll
                for (int c = 0; c < kAtKeys; ++c) s[c] = c >= from ? s[c] : -INFINITY;
            }
            const float by = GEN ? 1.f : p.scale_log2;
            float m4[4] = {mx, -INFINITY, -INFINITY, -INFINITY};  // (the factor is not negative, so it may follow the maximum)
#pragma unroll
            for (int c = 0; c < kAtKeys; ++c) m4[c & 3] = fmaxf(m4[c & 3], s[c]);
            const float m = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])), off = m * by;
            f = fast_exp2(mx * by - off);
            mx = m;
            float add = 0.f;
#pragma unroll
            for (int c = 0; c < kAtKeys; c += 8) {
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    s[c + e] = fast_exp2(GEN ? s[c + e] - off : fmaf(s[c + e], by, -off));
                    add += s[c + e];
                }
                *reinterpret_cast<uint4*>(prow + (c >> 3) * 128) = lb_pack_chunk<__nv_bfloat16>(s + c);
            }
            sum = fmaf(sum, f, add);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        lb_tc_fence_before();
        lb_mbar_arrive(&bar_p);
        if (tid == 0) {  // every row's weights are in shared memory, S_j and O_(j-1) have left tensor memory
            if (!lb_mbar_wait_bounded(&bar_p, (uint32_t)(j & 1), kTcWaitLimit) || !lb_mbar_wait_bounded(&bar_v[j & 1], (uint32_t)((j >> 1) & 1), kTcWaitLimit)) {
                failed = true;
            } else {
                lb_tc_fence_after();
                for (int k = 0; k < kAtKeys / 16; ++k)
                    lb_mma_f16(tmem + kAtKeys, lb_smem_desc(a_p + k * 256, 128, 1024), lb_smem_desc(a_v + (j & 1) * kVStage + k * 256, 128, 1024), id_o, k > 0 ? 1u : 0u);
                lb_mma_commit(&bar_o);
                if (j + 1 < ntiles) {
                    if (lb_mbar_wait_bounded(&bar_k[(j + 1) & 1], (uint32_t)(((j + 1) >> 1) & 1), kTcWaitLimit))
                        scores(j + 1);
                    else
                        failed = true;
                }
            }
        }
        __syncwarp();
        if (!lb_mbar_wait_bounded(&bar_o, (uint32_t)(j & 1), kTcWaitLimit)) failed = true;
        if (__any_sync(0xffffffffu, failed)) {
            failed = true;
            break;
        }
        if (tid == 0 && j + 2 < ntiles) load(j + 2);  // S_j and O_j are done: their stage is free
        __syncwarp();
        lb_tc_fence_after();
        constexpr int VS = VC % 64 == 0 ? 64 : VC % 32 == 0 ? 32 : 16;  // columns per wait
#pragma unroll
        for (int c = 0; c < VC; c += VS) {
            float v[VS];
#pragma unroll
            for (int e = 0; e < VS; e += 16) lb_tmem_ld16(tmem + lanes + kAtKeys + c + e, v + e);
            lb_tmem_wait_ld();
#pragma unroll
            for (int e = 0; e < VS; ++e) o[c + e] = fmaf(o[c + e], f, v[e]);
        }
    }
    if (failed) {
        if (lane == 0) atomicExch(p.status, 3);
    } else if (tok < p.T) {
        float r = __fdiv_rn(1.f, sum);
        if (GEN && p.gate) r *= lb_sigmoidf(p.gate[(size_t)tok * p.ldg + h]);
#pragma unroll
        for (int c = 0; c < VC; c += 8) {
            if (c < p.vdim) {
                float v[8];
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = o[c + e] * r;
                if (!GEN || p.vdim % 8 == 0) {
                    lb_img_store8<__nv_bfloat16>(p.out, tok, h * p.vdim + c, p.out_slices, v);
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const int col = h * p.vdim + c + e;
                        if (c + e < p.vdim) reinterpret_cast<__nv_bfloat16*>(p.out + lb_img_chunk(tok, col >> 3, p.out_slices))[col & 7] = __float2bfloat16_rn(v[e]);
                    }
                }
            }
        }
    }
    lb_tc_fence_before();
    __syncthreads();
    if (warp == 0) {
        lb_tc_fence_after();
        lb_tmem_dealloc(tmem, kTmem);
    }
}

template <int VC>
int launch(loom_b200_ctx* ctx, const LbAttnBlock& p) {
    const size_t smem = (size_t)p.dchunks * (2048 + 2 * 1024) + 2 * VC * 128 + 16384;
    const dim3 grid(p.heads, lb_ceil_div(p.T, 128));
    if (p.general) {
        LB_BIG_SMEM(ctx, (lb_attn_block_kernel<VC, true>), 220 * 1024);
        LB_LAUNCH(ctx, (lb_attn_block_kernel<VC, true>), grid, dim3(kAtThreads), smem, p);
    } else {
        LB_BIG_SMEM(ctx, (lb_attn_block_kernel<VC, false>), 220 * 1024);
        LB_LAUNCH(ctx, (lb_attn_block_kernel<VC, false>), grid, dim3(kAtThreads), smem, p);
    }
    return 0;
}

}  // namespace

int lb_attn_block(loom_b200_ctx* ctx, const LbAttnBlock& pin) {
    LbAttnBlock p = pin;
    p.status = ctx->status_dev;
    LB_REQUIRE(ctx, p.T > 0 && p.dchunks > 0 && p.dchunks % 2 == 0 && p.dchunks <= 32 && p.vrows % 8 == 0 && p.vdim <= p.vrows && p.vrows <= 128, "attention block: %d chunks, %d value rows",
               p.dchunks, p.vrows);
    LB_REQUIRE(ctx, !p.general || (p.ring >= 128 && p.ring % 128 == 0 && p.heads % p.kv_heads == 0), "attention block: ring of %d positions", p.ring);
    if (p.vrows <= 16) return launch<16>(ctx, p);
    if (p.vrows <= 32) return launch<32>(ctx, p);
    if (p.vrows <= 64) return launch<64>(ctx, p);
    if (p.vrows <= 96) return launch<96>(ctx, p);
    return launch<128>(ctx, p);
}
