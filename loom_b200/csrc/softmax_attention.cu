// softmax_attention.cu -- softmax attention over cached keys and values of grouped heads, with any of: unit-variance queries and
// keys, a learned bias by distance, chunks, a sink, a gate per head.  Storing a block of tokens, the step of one token per sequence
// (any precision), and the block's operands for the tensor-core kernel (attention_block.cu).
#include "mixers.cuh"

#include <cmath>

namespace {

constexpr int kTile = 64;  // positions of a tile: half of a block of keys; one K slice (two in 32-bit) of the transposed values
constexpr int kStepThreads = 256;

__host__ __device__ inline int vrows_of(int vdim) { return lb_round_up(vdim, 8); }

// 1 / root mean square of a head's row (a warp)
__device__ __forceinline__ float head_rstd(const float* row, int n, float eps, int lane) {
    float ss = 0.f;
    for (int d = lane; d < n; d += 32) ss = fmaf(row[d], row[d], ss);
    ss = lb_warp_sumf(ss);
    return __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)n), eps)));
}

// byte offset of 16-byte chunk c of a position's row of kv head g
__device__ __forceinline__ size_t key_chunk(int row, int g, int kv_heads, int kchunks, int c) {
    return ((size_t)(row >> 7) * kv_heads + g) * kchunks * 2048 + (size_t)((row & 127) >> 3) * kchunks * 128 + (size_t)c * 128 + (size_t)(row & 7) * 16;
}
template <typename WT>
__device__ __forceinline__ size_t value_at(int g, int v, int vrows, int row, int slices) {  // one element
    constexpr int C = LbElem<WT>::kChunk;
    return lb_img_chunk(g * vrows + v, row / C, slices) + (size_t)(row % C) * sizeof(WT);
}

// Queries (per-head blocks for the tensor-core kernel) and keys: a warp per (token, head), heads in blockIdx.y.  Values: the last rows
// of CTAs, a thread per value row and eight aligned positions.
template <typename WT>
__global__ void __launch_bounds__(256) lb_attention_store_kernel(const LbAttention p, int T, int kchunks, int qchunks, uint8_t* __restrict__ q_img, int rows, bool vec) {
    constexpr int C = LbElem<WT>::kChunk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, first = (p.pos0 & ~7) + (int)blockIdx.x * 8;
    const int QD = p.heads * p.dim, KD = p.kv_heads * p.dim, vrows = vrows_of(p.vdim);
    if ((int)blockIdx.y < rows) {
        const int i = (int)blockIdx.y + (q_img ? 0 : p.heads), pos = first + warp, t = pos - p.pos0;
        if (t < 0 || t >= T) return;
        const bool key = i >= p.heads;
        const int h = key ? i - p.heads : i;
        const float* x = p.proj + (size_t)t * p.ldp + (key ? QD + h * p.dim : h * p.dim);
        constexpr int KEEP = 8;  // columns of a lane that stay in registers: a pair of float4 for 256 channels
        float f[KEEP], by = 1.f;
        const int c0 = lane * KEEP;
        lb_load_cols<KEEP>(x, c0, p.dim, vec, f);  // (zero behind the last channel)
        if (p.qk_norm) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < KEEP; ++e) ss = fmaf(f[e], f[e], ss);
            for (int d = 32 * KEEP + lane; d < p.dim; d += 32) ss = fmaf(x[d], x[d], ss);
            ss = lb_warp_sumf(ss);
            by = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.dim), p.eps)));
        }
        uint8_t* kc = p.k + (size_t)p.lane0 * p.k_lane;
        const int r = pos % p.ring;
        for (int c = c0;; c += 32 * KEEP) {
#pragma unroll
            for (int e = 0; e < KEEP; ++e) f[e] *= by;
            if (key) {
#pragma unroll
                for (int e = 0; e < KEEP; e += C)
                    if ((c + e) / C < kchunks) *reinterpret_cast<uint4*>(kc + key_chunk(r, h, p.kv_heads, kchunks, (c + e) / C)) = lb_pack_chunk<WT>(f + e);
            } else if (c / 8 < qchunks) {
                *reinterpret_cast<uint4*>(q_img + key_chunk(t, h, p.heads, qchunks, c / 8)) = lb_pack_chunk<__nv_bfloat16>(f);
            }
            if (c + 32 * KEEP >= lb_round_up(p.dim, 16)) break;
            lb_load_cols<KEEP>(x, c + 32 * KEEP, p.dim, vec, f);
        }
        return;
    }
    uint8_t* vc = p.vt + (size_t)p.lane0 * p.vt_lane;
    const int t0 = first - p.pos0, r0 = first % p.ring, i = ((int)blockIdx.y - rows) * 256 + threadIdx.x;
    if (i >= p.kv_heads * p.vdim) return;
    const int g = i / p.vdim, v = i - g * p.vdim;
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = t0 + e >= 0 && t0 + e < T ? p.proj[(size_t)(t0 + e) * p.ldp + QD + KD + i] : 0.f;
    if (t0 >= 0 && t0 + 8 <= T) {
#pragma unroll
        for (int e = 0; e < 8; e += C) *reinterpret_cast<uint4*>(vc + lb_img_chunk(g * vrows + v, (r0 + e) / C, p.slices)) = lb_pack_chunk<WT>(f + e);
    } else {  // the eight positions hold tokens of other calls too
#pragma unroll
        for (int e = 0; e < 8; ++e)
            if (t0 + e >= 0 && t0 + e < T) *reinterpret_cast<WT*>(vc + value_at<WT>(g, v, vrows, r0 + e, p.slices)) = (WT)f[e];
    }
}

// ---- the step: one token per sequence ----------------------------------------------------------------------------------------
//
// CTA = (split of the visible positions, HB query heads of a kv head, token).  The split with the newest position takes its key and
// value from the projections and puts them into the cache.  Partial results are [token][kv head and block][split][HB] {vdim sums,
// maximum, sum}; the last CTA of a (token, heads) to arrive merges them, nothing waits.

// where the CTA works
struct StepPlace {
    int split, g, hb, m, h0, nh, pos, seq, low, active, j0, j1;
    bool newest;  // (otherwise every position is in the cache)
};
template <int HB>
__device__ __forceinline__ StepPlace step_place(const LbAttention& p, int splits) {
    StepPlace w;
    const int per = p.heads / p.kv_heads, nb = lb_ceil_div(per, HB);
    w.split = blockIdx.x;
    w.g = blockIdx.y / nb;
    w.hb = blockIdx.y % nb;
    w.m = blockIdx.z;
    w.h0 = w.g * per + w.hb * HB;
    w.nh = min(HB, per - w.hb * HB);
    w.pos = p.pos ? p.pos[w.m] : p.pos0 + w.m;
    w.seq = p.pos ? p.lane0 + w.m : p.lane0;
    w.low = p.chunk ? w.pos - w.pos % p.chunk : 0;
    const int first = w.low / kTile, ntiles = w.pos / kTile - first + 1;  // every tile has a visible position
    w.active = min(splits, ntiles);
    w.j0 = first + (int)((long long)ntiles * w.split / w.active);
    w.j1 = first + (int)((long long)ntiles * (w.split + 1) / w.active);
    w.newest = p.pos && w.split == w.active - 1;
    return w;
}

__device__ __forceinline__ float* partial_row(const LbAttention& p, float* part, int group, int splits, int split, int HB) {
    return part + ((size_t)group * splits + split) * HB * (p.vdim + 2);
}

// after every thread of the CTA has written its part of the partial result; sw: HB * 64 floats
template <int HB>
__device__ __forceinline__ void merge_splits(const LbAttention& p, float* part, unsigned* count, int group, int splits, int active, int h0, int nh, const float* gate, float* sw,
                                             float* o) {
    __shared__ bool s_last;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, row = p.vdim + 2;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        s_last = atomicAdd(count + group, 1u) == (unsigned)active - 1;
        if (s_last) count[group] = 0;
    }
    __syncthreads();
    if (!s_last) return;
    __threadfence();
    const float* all = partial_row(p, part, group, splits, 0, HB);
    for (int h = warp; h < nh; h += 8) {
        float mx = -INFINITY, den = 0.f, top[2], sum[2];  // (at most 64 splits)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int s = lane + 32 * i;
            top[i] = s < active ? __ldcg(all + ((size_t)s * HB + h) * row + p.vdim) : -INFINITY;
            sum[i] = s < active ? __ldcg(all + ((size_t)s * HB + h) * row + p.vdim + 1) : 0.f;
            mx = fmaxf(mx, top[i]);
        }
        mx = lb_warp_max(mx);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            top[i] = expf(top[i] - mx);
            den = fmaf(top[i], sum[i], den);
        }
        den = lb_warp_sumf(den);
        float r = __fdiv_rn(1.f, den);
        if (p.head_gate) r *= lb_sigmoidf(gate[h0 + h]);
        sw[h * 64 + lane] = top[0] * r;
        sw[h * 64 + lane + 32] = top[1] * r;
    }
    __syncthreads();
    for (int i = tid; i < nh * p.vdim; i += kStepThreads) {
        const int h = i / p.vdim, v = i - h * p.vdim;
        float a = 0.f;
#pragma unroll 8
        for (int s = 0; s < active; ++s) a = fmaf(sw[h * 64 + s], __ldcg(all + ((size_t)s * HB + h) * row + v), a);
        o[(h0 + h) * p.vdim + v] = a;
    }
}

// Any precision and head size, plain multiply-adds.  Tiles of 64 positions: four threads per key for the scores, a warp per head for the
// running softmax, then four threads per value row and K slice for the weighted sum.
template <typename WT, int HB>
__global__ void __launch_bounds__(kStepThreads) lb_attention_step_kernel(const LbAttention p, int kchunks, int splits, float* __restrict__ part, unsigned* __restrict__ count,
                                                                         float* __restrict__ out, int ldo) {
    extern __shared__ __align__(16) uint8_t sm[];
    constexpr int C = LbElem<WT>::kChunk, S = LbElem<WT>::kSlice, KS = kTile / S;  // KS: K slices of a tile
    __shared__ __align__(16) float s_w[HB][kTile];
    __shared__ float s_max[HB], s_sum[HB], s_fac[HB], s_new[HB], s_rq[HB], s_rk;
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const StepPlace w = step_place<HB>(p, splits);
    const int split = w.split, g = w.g, hb = w.hb, m = w.m, h0 = w.h0, nh = w.nh, pos = w.pos, seq = w.seq, low = w.low, active = w.active, j0 = w.j0, j1 = w.j1;
    const bool newest = w.newest;
    if (split >= active) return;
    const int vrows = vrows_of(p.vdim), QD = p.heads * p.dim, KD = p.kv_heads * p.dim, kcols = kchunks * C;
    float *sq = reinterpret_cast<float*>(sm), *so = sq + HB * kcols;              // queries [HB][kcols]; sums [HB][vrows]
    uint4* skey = reinterpret_cast<uint4*>(so + HB * vrows);                      // the newest key's chunks
    float* sval = reinterpret_cast<float*>(skey + kchunks);                       // the newest value
    const float* row = p.proj + (size_t)m * p.ldp;
    uint8_t *kc = p.k + (size_t)seq * p.k_lane, *vc = p.vt + (size_t)seq * p.vt_lane;
    for (int i = warp; i <= nh; i += 8) {
        const float* x = i < nh ? row + (h0 + i) * p.dim : row + QD + g * p.dim;
        const float by = p.qk_norm ? head_rstd(x, p.dim, p.eps, lane) : 1.f;
        if (lane == 0) (i < nh ? s_rq[i] : s_rk) = by;
    }
    if (tid < HB) {
        s_max[tid] = p.sink && split == 0 ? 0.f : -INFINITY;
        s_sum[tid] = p.sink && split == 0 ? 1.f : 0.f;
    }
    for (int i = tid; i < HB * vrows; i += kStepThreads) so[i] = 0.f;
    __syncthreads();
    for (int i = tid; i < HB * kcols; i += kStepThreads) {
        const int h = i / kcols, d = i - h * kcols;
        sq[i] = h < nh && d < p.dim ? row[(h0 + h) * p.dim + d] * s_rq[h] : 0.f;
    }
    if (newest) {
        const int r = pos % p.ring;
        for (int c = tid; c < kchunks; c += kStepThreads) {
            float f[C];
            lb_load_cols<C>(row + QD + g * p.dim, c * C, p.dim, false, f);
#pragma unroll
            for (int e = 0; e < C; ++e) f[e] *= s_rk;
            const uint4 w = lb_pack_chunk<WT>(f);
            skey[c] = w;
            if (hb == 0) *reinterpret_cast<uint4*>(kc + key_chunk(r, g, p.kv_heads, kchunks, c)) = w;
        }
        for (int v = tid; v < p.vdim; v += kStepThreads) {
            const WT w = (WT)row[QD + KD + g * p.vdim + v];
            sval[v] = (float)w;
            if (hb == 0) *reinterpret_cast<WT*>(vc + value_at<WT>(g, v, vrows, r, p.slices)) = w;
        }
    }
    __syncthreads();
    const int kg = (warp << 3) | (lane >> 2), kt = lane & 3;  // key of the tile, quarter of its chunks
    for (int j = j0; j < j1; ++j) {
        const int base = j * kTile, rbase = base % p.ring;
        // ---- scores ----
        {
            const int key = base + kg;
            float a[HB];
#pragma unroll
            for (int h = 0; h < HB; ++h) a[h] = 0.f;
            if (key >= low && key <= pos) {
                const uint8_t* src = kc + key_chunk(rbase + kg, g, p.kv_heads, kchunks, 0);
                const bool fresh = newest && key == pos;
#pragma unroll 4
                for (int c = kt; c < kchunks; c += 4) {
                    float f[C];
                    lb_unpack_chunk<WT>(fresh ? skey[c] : *reinterpret_cast<const uint4*>(src + (size_t)c * 128), f);
#pragma unroll
                    for (int h = 0; h < HB; ++h)
#pragma unroll
                        for (int e = 0; e < C; e += 4) {
                            const float4 q = *reinterpret_cast<const float4*>(sq + h * kcols + c * C + e);
                            a[h] = fmaf(f[e], q.x, fmaf(f[e + 1], q.y, fmaf(f[e + 2], q.z, fmaf(f[e + 3], q.w, a[h]))));
                        }
                }
            }
            const float* bias = p.bias + kBiasFront + min(max(pos - key, 0), p.bias_len - 1);
#pragma unroll
            for (int h = 0; h < HB; ++h) {
                a[h] += __shfl_xor_sync(0xffffffffu, a[h], 1);
                a[h] += __shfl_xor_sync(0xffffffffu, a[h], 2);
                if (kt == 0) {
                    float s = -INFINITY;
                    if (h < nh && key >= low && key <= pos) s = fmaf(a[h], p.scale, p.bias ? bias[(size_t)(h0 + h) * p.bias_ld] : 0.f);
                    s_w[h][kg] = s;
                }
            }
        }
        __syncthreads();
        // ---- running softmax: a warp per head, two positions per lane (every tile has a visible position) ----
        for (int h = warp; h < nh; h += 8) {
            const float x0 = s_w[h][lane], x1 = s_w[h][lane + 32], old = s_max[h];
            const float mx = fmaxf(old, lb_warp_max(fmaxf(x0, x1)));
            const float w0 = expf(x0 - mx), w1 = expf(x1 - mx), sum = lb_warp_sumf(w0 + w1);
            const int at = newest && pos >= base && pos < base + kTile ? pos - base : -1;  // its value is not in the cache yet
            s_w[h][lane] = lane == at ? 0.f : w0;
            s_w[h][lane + 32] = lane + 32 == at ? 0.f : w1;
            if (at >= 0 && lane == (at & 31)) s_new[h] = at < 32 ? w0 : w1;
            if (lane == 0) {
                const float f = expf(old - mx);
                s_max[h] = mx;
                s_sum[h] = fmaf(s_sum[h], f, sum);
                s_fac[h] = f;
            }
        }
        __syncthreads();
        // ---- weighted sum: lane (row of eight, chunk quarter) ----
        const bool with_new = newest && pos >= base && pos < base + kTile;
        for (int vg = warp; vg < vrows / 8; vg += 8) {
            const int v = vg * 8 + (lane >> 2), irow = g * vrows + v;
            uint4 w[2 * KS];
#pragma unroll
            for (int x = 0; x < 2 * KS; ++x) {
                const int c = kt + 4 * x;
                w[x] = *reinterpret_cast<const uint4*>(vc + lb_img_chunk(irow, rbase / C + c, p.slices));
            }
            float a[HB];
#pragma unroll
            for (int h = 0; h < HB; ++h) a[h] = 0.f;
#pragma unroll
            for (int x = 0; x < 2 * KS; ++x) {
                const int c = kt + 4 * x;
                float f[C];
                lb_unpack_chunk<WT>(w[x], f);
#pragma unroll
                for (int h = 0; h < HB; ++h)
#pragma unroll
                    for (int e = 0; e < C; e += 4) {
                        const float4 s = *reinterpret_cast<const float4*>(&s_w[h][c * C + e]);
                        a[h] = fmaf(f[e], s.x, fmaf(f[e + 1], s.y, fmaf(f[e + 2], s.z, fmaf(f[e + 3], s.w, a[h]))));
                    }
            }
#pragma unroll
            for (int h = 0; h < HB; ++h) {
                a[h] += __shfl_xor_sync(0xffffffffu, a[h], 1);
                a[h] += __shfl_xor_sync(0xffffffffu, a[h], 2);
                if (kt == 0 && h < nh) {
                    if (with_new && v < p.vdim) a[h] = fmaf(s_new[h], sval[v], a[h]);
                    so[h * vrows + v] = fmaf(so[h * vrows + v], s_fac[h], a[h]);
                }
            }
        }
        __syncthreads();
    }
    const float* gate = row + QD + KD + p.kv_heads * p.vdim;
    float* o = out + (size_t)m * ldo;
    const int group = m * gridDim.y + blockIdx.y;
    if (active == 1) {
        for (int i = tid; i < nh * p.vdim; i += kStepThreads) {
            const int h = i / p.vdim, v = i - h * p.vdim;
            const float r = __fdiv_rn(so[h * vrows + v], s_sum[h]);
            o[(h0 + h) * p.vdim + v] = p.head_gate ? r * lb_sigmoidf(gate[h0 + h]) : r;
        }
        return;
    }
    float* mine = partial_row(p, part, group, splits, split, HB);
    for (int i = tid; i < nh * p.vdim; i += kStepThreads) {
        const int h = i / p.vdim, v = i - h * p.vdim;
        mine[h * (p.vdim + 2) + v] = so[h * vrows + v];
    }
    if (tid < nh) {
        mine[tid * (p.vdim + 2) + p.vdim] = s_max[tid];
        mine[tid * (p.vdim + 2) + p.vdim + 1] = s_sum[tid];
    }
    merge_splits<HB>(p, part, count, group, splits, active, h0, nh, gate, sq, o);
}

__device__ __forceinline__ void mma_bf16(float* d, uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
// 16 rows x one 16-byte chunk per lane column: which k of a chunk an MMA takes is the same for both operands, so the order cancels
__device__ __forceinline__ void mma_chunk(float* d, const uint4& a0, const uint4& a1, const uint4& b) {
    mma_bf16(d, a0.x, a1.x, a0.y, a1.y, b.x, b.y);
    mma_bf16(d, a0.z, a1.z, a0.w, a1.w, b.z, b.w);
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

// bf16, up to sixteen query heads of a kv head per CTA on the tensor cores (MMA rows that no head uses cost nothing that is scarce here):
// keys and values go from global memory straight into the B fragments.  A warp has eight of a tile's 64 keys for the scores and every
// eighth group of eight value rows for the weighted sum; queries and softmax weights are bf16 pairs.  The next tile's keys and values
// are requested as soon as this tile's fragments have been used.
constexpr int kMmaHeads = 16;

template <int NK, int NG>  // key chunks per lane (dim <= 32 NK), groups of value rows per warp (vdim <= 64 NG)
__global__ void __launch_bounds__(kStepThreads, 2) lb_attention_step_mma_kernel(const LbAttention p, int kchunks, int splits, float* __restrict__ part, unsigned* __restrict__ count,
                                                                                float* __restrict__ out, int ldo) {
    constexpr int HB = kMmaHeads, SL = kTile + 4;
    __shared__ __align__(16) uint4 s_q[2][NK * 4][HB + 2], s_key[NK * 4], s_p[2][kTile / 8][HB + 2];  // (rows padded against bank conflicts)
    __shared__ __align__(16) float s_s[HB][SL];  // (the merge uses 64 a head)
    __shared__ float s_max[HB], s_sum[HB], s_fac[HB];
    __shared__ __nv_bfloat16 s_val[NG * 64];
    lb_pdl_launch_dependents();
    lb_pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const StepPlace w = step_place<HB>(p, splits);
    if (w.split >= w.active) return;
    const int vrows = vrows_of(p.vdim), QD = p.heads * p.dim, KD = p.kv_heads * p.dim;
    const float* row = p.proj + (size_t)w.m * p.ldp;
    uint8_t *kc = p.k + (size_t)w.seq * p.k_lane, *vc = p.vt + (size_t)w.seq * p.vt_lane;
    uint4 kr[NK], vr[NG][2];
    auto load_keys = [&](int j) {
        const uint8_t* src = kc + key_chunk((j * kTile) % p.ring + warp * 8 + g, w.g, p.kv_heads, kchunks, 0);
#pragma unroll
        for (int i = 0; i < NK; ++i)
            if (4 * i + t < kchunks) kr[i] = *reinterpret_cast<const uint4*>(src + (size_t)(4 * i + t) * 128);
    };
    auto load_values = [&](int j) {
        const int c0 = (j * kTile) % p.ring / 8;
#pragma unroll
        for (int i = 0; i < NG; ++i)
            if ((warp + 8 * i) * 8 < vrows)
#pragma unroll
                for (int x = 0; x < 2; ++x) vr[i][x] = *reinterpret_cast<const uint4*>(vc + lb_img_chunk(w.g * vrows + (warp + 8 * i) * 8 + g, c0 + t + 4 * x, p.slices));
    };
#pragma unroll
    for (int i = 0; i < NK; ++i) kr[i] = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < NG; ++i) vr[i][0] = vr[i][1] = make_uint4(0, 0, 0, 0);
    load_keys(w.j0);
    load_values(w.j0);
    // queries, and the newest key, a warp per row and eight columns per lane
    for (int i = warp; i < HB + (w.newest ? 1 : 0); i += 8) {
        const bool key = i == HB;
        const float* x = key ? row + QD + w.g * p.dim : row + (w.h0 + i) * p.dim;
        float f[8], by = key || i < w.nh ? 1.f : 0.f;
        if (by != 0.f) {
            lb_load_cols<8>(x, lane * 8, p.dim, false, f);
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] = 0.f;
        }
        if (p.qk_norm && by != 0.f) {
            float ss = 0.f;
#pragma unroll
            for (int e = 0; e < 8; ++e) ss = fmaf(f[e], f[e], ss);
            ss = lb_warp_sumf(ss);
            by = __fdiv_rn(1.f, sqrtf(__fadd_rn(__fdiv_rn(ss, (float)p.dim), p.eps)));
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] *= by;
        if (lane >= NK * 4) continue;
        if (!key) {
            split_bf16(f, s_q[0][lane][i], s_q[1][lane][i]);
        } else {
            s_key[lane] = lb_pack_chunk<__nv_bfloat16>(f);
            if (w.hb == 0 && lane < kchunks) *reinterpret_cast<uint4*>(kc + key_chunk(w.pos % p.ring, w.g, p.kv_heads, kchunks, lane)) = s_key[lane];
        }
    }
    if (w.newest)
        for (int v = tid; v < p.vdim; v += kStepThreads) {
            const __nv_bfloat16 x = __float2bfloat16_rn(row[QD + KD + w.g * p.vdim + v]);
            s_val[v] = x;
            if (w.hb == 0) *reinterpret_cast<__nv_bfloat16*>(vc + value_at<__nv_bfloat16>(w.g, v, vrows, w.pos % p.ring, p.slices)) = x;
        }
    if (tid < HB) {
        s_max[tid] = p.sink && w.split == 0 ? 0.f : -INFINITY;
        s_sum[tid] = p.sink && w.split == 0 ? 1.f : 0.f;
    }
    float o[NG][4];
#pragma unroll
    for (int i = 0; i < NG; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    __syncthreads();
    for (int j = w.j0; j < w.j1; ++j) {
        const int base = j * kTile, at = w.newest && w.pos / kTile == j ? w.pos - base : -1;  // the newest position's place in the tile
        // ---- scores of keys warp * 8 + 0..7 ----
        {
            float bias[4] = {0.f, 0.f, 0.f, 0.f}, d[4] = {0.f, 0.f, 0.f, 0.f};
            const int key0 = base + warp * 8 + 2 * t;  // d: heads g (0, 1) and g + 8 (2, 3), keys key0 and key0 + 1
            if (p.bias)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int h = g + 8 * (e >> 1), dist = min(max(w.pos - key0 - (e & 1), 0), p.bias_len - 1);
                    if (h < w.nh) bias[e] = __ldg(p.bias + (size_t)(w.h0 + h) * p.bias_ld + kBiasFront + dist);
                }
            if (at >= 0 && warp * 8 + g == at)
#pragma unroll
                for (int i = 0; i < NK; ++i)
                    if (4 * i + t < kchunks) kr[i] = s_key[4 * i + t];
#pragma unroll
            for (int i = 0; i < NK; ++i)
#pragma unroll
                for (int half = 0; half < 2; ++half) mma_chunk(d, s_q[half][4 * i + t][g], s_q[half][4 * i + t][g + 8], kr[i]);
            if (j + 1 < w.j1) load_keys(j + 1);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = key0 + (e & 1);
                s_s[g + 8 * (e >> 1)][warp * 8 + 2 * t + (e & 1)] = key >= w.low && key <= w.pos ? fmaf(d[e], p.scale, bias[e]) : -INFINITY;
            }
        }
        __syncthreads();
        // ---- running softmax: sixteen threads per head, four positions each ----
        {
            const int h = tid >> 4, q = tid & 15;
            const float4 x = *reinterpret_cast<const float4*>(&s_s[h][q * 4]);
            float mx = fmaxf(fmaxf(x.x, x.y), fmaxf(x.z, x.w));
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
            const float old = s_max[h], nm = fmaxf(old, mx);
            float e[4] = {expf(x.x - nm), expf(x.y - nm), expf(x.z - nm), expf(x.w - nm)}, sum = (e[0] + e[1]) + (e[2] + e[3]);
#pragma unroll
            for (int off = 8; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
            __syncwarp();
            if (q == 0) {
                const float f = expf(old - nm);
                s_max[h] = nm;
                s_fac[h] = f;
                s_sum[h] = fmaf(s_sum[h], f, sum);
            }
            float l[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float hi = __bfloat162float(__float2bfloat16_rn(e[i]));
                l[i] = e[i] - hi;
                e[i] = hi;
            }
            *(reinterpret_cast<uint2*>(&s_p[0][q >> 1][h]) + (q & 1)) = make_uint2(lb_pack_bf16(e[0], e[1]), lb_pack_bf16(e[2], e[3]));
            *(reinterpret_cast<uint2*>(&s_p[1][q >> 1][h]) + (q & 1)) = make_uint2(lb_pack_bf16(l[0], l[1]), lb_pack_bf16(l[2], l[3]));
        }
        __syncthreads();
        // ---- weighted sum: chunk t + 4 x holds positions 8 (t + 4 x) ... of this lane's value rows ----
        {
            const float f0 = s_fac[g], f1 = s_fac[g + 8];
            if (at >= 0) {  // the newest position's values are not in the cache yet
                const int c = at >> 3;
#pragma unroll
                for (int i = 0; i < NG; ++i) {
                    const int v = (warp + 8 * i) * 8 + g;
                    const uint32_t put = (uint32_t)__bfloat16_as_ushort(s_val[v < p.vdim ? v : 0]) << (16 * (at & 1)), keep = ~(0xffffu << (16 * (at & 1)));
#pragma unroll
                    for (int x = 0; x < 2; ++x) {
                        const int word = c == t + 4 * x && v < p.vdim ? (at & 7) >> 1 : -1;
                        uint4& y = vr[i][x];
                        y.x = word == 0 ? (y.x & keep) | put : y.x;
                        y.y = word == 1 ? (y.y & keep) | put : y.y;
                        y.z = word == 2 ? (y.z & keep) | put : y.z;
                        y.w = word == 3 ? (y.w & keep) | put : y.w;
                    }
                }
            }
#pragma unroll
            for (int i = 0; i < NG; ++i) {
                o[i][0] *= f0;
                o[i][1] *= f0;
                o[i][2] *= f1;
                o[i][3] *= f1;
            }
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const uint4 a0 = s_p[half][t + 4 * x][g], a1 = s_p[half][t + 4 * x][g + 8];
#pragma unroll
                    for (int i = 0; i < NG; ++i) mma_chunk(o[i], a0, a1, vr[i][x]);
                }
            if (j + 1 < w.j1) load_values(j + 1);
        }
        __syncthreads();
    }
    const float* gate = row + QD + KD + p.kv_heads * p.vdim;
    float* dst = out + (size_t)w.m * ldo;
    const int group = w.m * gridDim.y + blockIdx.y;
    float* mine = partial_row(p, part, group, splits, w.split, HB);
#pragma unroll
    for (int hb = 0; hb < 2; ++hb) {
        const int h = g + 8 * hb;
        if (h >= w.nh) continue;
        const float r = w.active > 1 ? 1.f : __fdiv_rn(p.head_gate ? lb_sigmoidf(gate[w.h0 + h]) : 1.f, s_sum[h]);
        float* y = w.active > 1 ? mine + h * (p.vdim + 2) : dst + (w.h0 + h) * p.vdim;
#pragma unroll
        for (int i = 0; i < NG; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int v = (warp + 8 * i) * 8 + 2 * t + e;
                if (v < p.vdim) y[v] = o[i][2 * hb + e] * r;
            }
    }
    if (w.active == 1) return;
    if (tid < w.nh) {
        mine[tid * (p.vdim + 2) + p.vdim] = s_max[tid];
        mine[tid * (p.vdim + 2) + p.vdim + 1] = s_sum[tid];
    }
    merge_splits<HB>(p, part, count, group, splits, w.active, w.h0, w.nh, gate, &s_s[0][0], dst);
}

// query heads of a CTA of the step
int heads_block(const LbAttention& p) {
    const int per = p.heads / p.kv_heads;
    if (p.mma) return kMmaHeads;
    return per >= 8 ? 8 : per > 2 ? 4 : per;
}
int groups_of(const LbAttention& p) { return p.kv_heads * lb_ceil_div(p.heads / p.kv_heads, heads_block(p)); }

size_t step_smem(const LbAttention& p, int HB, int kchunks, int C) {
    const size_t front = (size_t)HB * kchunks * C < (size_t)HB * 64 ? (size_t)HB * 64 : (size_t)HB * kchunks * C;  // (the merge uses 64 a head)
    return (front + (size_t)HB * vrows_of(p.vdim)) * sizeof(float) + (size_t)kchunks * 16 + (size_t)p.vdim * sizeof(float);
}
constexpr size_t kStepSmem = 200 * 1024;

template <typename WT, int HB>
int launch_step(loom_b200_ctx* ctx, const LbAttention& p, int tokens, int kchunks, float* part, unsigned* count, float* out, int ldo) {
    const size_t smem = step_smem(p, HB, kchunks, LbElem<WT>::kChunk);
    LB_REQUIRE(ctx, smem <= kStepSmem, "attention: head dimensions %d and %d", p.dim, p.vdim);
    if (smem > 40 * 1024) LB_BIG_SMEM(ctx, (lb_attention_step_kernel<WT, HB>), kStepSmem);
    const int splits = lb_attention_splits(ctx, p, tokens);
    LB_LAUNCH(ctx, (lb_attention_step_kernel<WT, HB>), dim3(splits, groups_of(p), tokens), dim3(kStepThreads), smem, p, kchunks, splits, part, count, out, ldo);
    return 0;
}

template <typename WT>
int step_heads(loom_b200_ctx* ctx, const LbAttention& p, int tokens, int kchunks, float* part, unsigned* count, float* out, int ldo) {
    switch (heads_block(p)) {
        case 1: return launch_step<WT, 1>(ctx, p, tokens, kchunks, part, count, out, ldo);
        case 2: return launch_step<WT, 2>(ctx, p, tokens, kchunks, part, count, out, ldo);
        case 4: return launch_step<WT, 4>(ctx, p, tokens, kchunks, part, count, out, ldo);
    }
    return launch_step<WT, 8>(ctx, p, tokens, kchunks, part, count, out, ldo);
}

template <int NK, int NG>
int launch_mma(loom_b200_ctx* ctx, const LbAttention& p, int tokens, int kchunks, float* part, unsigned* count, float* out, int ldo) {
    const int splits = lb_attention_splits(ctx, p, tokens);
    LB_LAUNCH(ctx, (lb_attention_step_mma_kernel<NK, NG>), dim3(splits, groups_of(p), tokens), dim3(kStepThreads), 0, p, kchunks, splits, part, count, out, ldo);
    return 0;
}

}  // namespace

bool lb_attention_step_mma(int dim, int vdim, int dtype) { return dtype == LOOM_B200_DTYPE_BF16 && dim <= 256 && vdim <= 256; }

int lb_attention_kchunks(int dim, int dtype) { return lb_round_up(lb_ceil_div(dim, dtype == LOOM_B200_DTYPE_BF16 ? 8 : 4), 2); }

size_t lb_attention_k_bytes(int kv_heads, int dim, int ring, int dtype) { return (size_t)(ring / 128) * kv_heads * lb_attention_kchunks(dim, dtype) * 2048; }

size_t lb_attention_vt_bytes(int kv_heads, int vdim, int ring, int dtype) { return lb_img_bytes(kv_heads * vrows_of(vdim), ring, dtype); }

size_t lb_attention_q_bytes(const LbAttention& p, int rows) { return (size_t)lb_ceil_div(rows, 128) * p.heads * lb_attention_kchunks(p.dim, LOOM_B200_DTYPE_BF16) * 2048; }

int lb_attention_store(loom_b200_ctx* ctx, int dtype, const LbAttention& p, int T, uint8_t* q_img) {
    const int kch = lb_attention_kchunks(p.dim, dtype), qch = lb_attention_kchunks(p.dim, LOOM_B200_DTYPE_BF16);
    const int rows = p.kv_heads + (q_img && dtype == LOOM_B200_DTYPE_BF16 ? p.heads : 0);
    const dim3 grid((p.pos0 + T - 1) / 8 - p.pos0 / 8 + 1, rows + lb_ceil_div(p.kv_heads * p.vdim, 256));
    const bool vec = p.dim % 4 == 0 && lb_vec_rows(p.proj, p.ldp);
    if (dtype == LOOM_B200_DTYPE_BF16)
        LB_LAUNCH(ctx, lb_attention_store_kernel<__nv_bfloat16>, grid, dim3(256), 0, p, T, kch, qch, q_img, rows, vec);
    else
        LB_LAUNCH(ctx, lb_attention_store_kernel<float>, grid, dim3(256), 0, p, T, kch, qch, nullptr, rows, vec);
    return 0;
}

int lb_attention_splits(loom_b200_ctx* ctx, const LbAttention& p, int tokens) {
    int s = lb_ceil_div(4 * ctx->sm_count, groups_of(p) * tokens);
    const int tiles = (p.chunk && p.chunk < p.ring ? p.chunk : p.ring) / kTile + 2;  // a chunk may begin and end inside a tile
    if (s > tiles) s = tiles;
    if (s > 64) s = 64;
    return s < 1 ? 1 : s;
}

size_t lb_attention_part_elems(loom_b200_ctx* ctx, const LbAttention& p, int tokens) {
    return (size_t)tokens * groups_of(p) * lb_attention_splits(ctx, p, tokens) * heads_block(p) * (p.vdim + 2);
}

size_t lb_attention_counters(const LbAttention& p, int tokens) { return (size_t)tokens * groups_of(p); }

int lb_attention_step(loom_b200_ctx* ctx, int dtype, const LbAttention& p, int tokens, float* part, unsigned* count, float* out, int ldo) {
    const int kch = lb_attention_kchunks(p.dim, dtype);
    LB_REQUIRE(ctx, tokens > 0 && tokens <= 65535, "attention: %d tokens", tokens);
    if (p.mma) {
        const bool k4 = p.dim <= 128, v2 = p.vdim <= 128;
        if (k4) return v2 ? launch_mma<4, 2>(ctx, p, tokens, kch, part, count, out, ldo) : launch_mma<4, 4>(ctx, p, tokens, kch, part, count, out, ldo);
        return v2 ? launch_mma<8, 2>(ctx, p, tokens, kch, part, count, out, ldo) : launch_mma<8, 4>(ctx, p, tokens, kch, part, count, out, ldo);
    }
    return dtype == LOOM_B200_DTYPE_BF16 ? step_heads<__nv_bfloat16>(ctx, p, tokens, kch, part, count, out, ldo) : step_heads<float>(ctx, p, tokens, kch, part, count, out, ldo);
}

bool lb_attention_block_supported(const LbAttention& p) { return p.dim <= 256 && p.vdim <= 128; }

int lb_attention_block(loom_b200_ctx* ctx, const LbAttention& p, int T, const uint8_t* q_img, uint8_t* out, int out_slices) {
    LbAttnBlock a;
    a.q = q_img;
    a.k = p.k + (size_t)p.lane0 * p.k_lane;
    a.vt = p.vt + (size_t)p.lane0 * p.vt_lane;
    a.heads = p.heads;
    a.kv_heads = p.kv_heads;
    a.dchunks = lb_attention_kchunks(p.dim, LOOM_B200_DTYPE_BF16);
    a.vdim = p.vdim;
    a.vrows = vrows_of(p.vdim);
    a.vslices = p.slices;
    a.T = T;
    a.pos0 = p.pos0;
    a.scale_log2 = p.scale * 1.4426950408889634f;
    a.out = out;
    a.out_slices = out_slices;
    a.general = true;
    a.chunk = p.chunk;
    a.ring = p.ring;
    a.bias = p.bias_log2;
    a.bias_len = p.bias_len;
    a.bias_ld = p.bias_ld;
    a.sink = p.sink;
    a.gate = p.head_gate ? p.proj + (size_t)p.heads * p.dim + (size_t)p.kv_heads * (p.dim + p.vdim) : nullptr;
    a.ldg = p.ldp;
    return lb_attn_block(ctx, a);
}
