// dense.cuh -- matrices of 16-bit or 32-bit floats and the products the layer stacks (stack.cu) are made of: storage,
// the one-token-per-sequence GEMV with its fused prologues and epilogues, and the token-block GEMM.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

// ---- the block image ------------------------------------------------------------------------------------
//
// Weights, activations of a token block and the latent cache share one layout: 16 KB blocks of 128 rows x one K slice
// of 128 bytes (64 bf16 or 32 float columns), inside a block [row/8][16-byte chunk of the slice][row%8][16 B].  It is
// the K-major no-swizzle core-matrix image that tcgen05 reads from shared memory, so a pipeline stage is one bulk copy;
// a warp that loads chunks t = 0..3 of rows g = 0..7 reads 512 consecutive bytes, so the GEMV streams the same bytes
// without a second copy of the weights.  Rows and columns are padded with zeros.
constexpr int kImgRows = 128;
constexpr int kImgBlock = 16384;

template <typename WT>
struct LbElem {
    static constexpr int kChunk = 16 / (int)sizeof(WT);  // elements of a 16-byte chunk
    static constexpr int kSlice = 8 * kChunk;            // columns of a K slice
};

__host__ __device__ __forceinline__ int lb_ceil_div(int a, int b) { return (a + b - 1) / b; }
__host__ __device__ __forceinline__ int lb_round_up(int a, int b) { return lb_ceil_div(a, b) * b; }

// byte offset of 16-byte chunk c of a row in an image of `slices` K slices
__host__ __device__ __forceinline__ size_t lb_img_chunk(int row, int chunk, int slices) {
    return ((size_t)(row >> 7) * slices + (chunk >> 3)) * kImgBlock + (size_t)((row & 127) >> 3) * 1024 + (size_t)(chunk & 7) * 128 +
           (size_t)(row & 7) * 16;
}

static inline int lb_slice_cols(int dtype) { return dtype == LOOM_B200_DTYPE_BF16 ? 64 : 32; }
static inline int lb_slices_of(int cols, int dtype) { return lb_ceil_div(cols, lb_slice_cols(dtype)); }
static inline size_t lb_img_bytes(int rows, int cols, int dtype) {
    return (size_t)lb_ceil_div(rows, kImgRows) * lb_slices_of(cols, dtype) * kImgBlock;
}

struct loom_b200_matrix {
    int rows = 0, cols = 0, groups = 1;  // `groups` matrices of one shape in one allocation (the experts of a layer)
    int dtype = 0;
    int slices = 0, device = 0;
    size_t group_bytes = 0;
    uint8_t* data = nullptr;
};

// ---- device helpers ---------------------------------------------------------------------------------------

template <typename WT>
__device__ __forceinline__ void lb_unpack_chunk(const uint4& c, float* f);
template <>
__device__ __forceinline__ void lb_unpack_chunk<float>(const uint4& c, float* f) {
    f[0] = __uint_as_float(c.x);
    f[1] = __uint_as_float(c.y);
    f[2] = __uint_as_float(c.z);
    f[3] = __uint_as_float(c.w);
}
template <>
__device__ __forceinline__ void lb_unpack_chunk<__nv_bfloat16>(const uint4& c, float* f) {
    const uint32_t w[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(w[i] << 16);
        f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ uint32_t lb_pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t*>(&v);
}
template <typename WT>
__device__ __forceinline__ uint4 lb_pack_chunk(const float* f);
template <>
__device__ __forceinline__ uint4 lb_pack_chunk<float>(const float* f) {
    return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
}
template <>
__device__ __forceinline__ uint4 lb_pack_chunk<__nv_bfloat16>(const float* f) {
    return make_uint4(lb_pack_bf16(f[0], f[1]), lb_pack_bf16(f[2], f[3]), lb_pack_bf16(f[4], f[5]), lb_pack_bf16(f[6], f[7]));
}
// stores eight consecutive columns (first column a multiple of eight) of an image row
template <typename WT>
__device__ __forceinline__ void lb_img_store8(uint8_t* img, int row, int col0, int slices, const float* f) {
    constexpr int C = LbElem<WT>::kChunk;
#pragma unroll
    for (int i = 0; i < 8 / C; ++i)
        *reinterpret_cast<uint4*>(img + lb_img_chunk(row, col0 / C + i, slices)) = lb_pack_chunk<WT>(f + i * C);
}

// C floats of a row from column k on, zero from column n on; vec: the row starts on a 16-byte boundary
template <int C>
__device__ __forceinline__ void lb_load_cols(const float* row, int k, int n, bool vec, float* f) {
    if (vec && k + C <= n) {
#pragma unroll
        for (int i = 0; i < C; i += 4) {
            const float4 v = *reinterpret_cast<const float4*>(row + k + i);
            f[i] = v.x;
            f[i + 1] = v.y;
            f[i + 2] = v.z;
            f[i + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < C; ++i) f[i] = k + i < n ? row[k + i] : 0.f;
    }
}
static inline bool lb_vec_rows(const float* p, int ld) { return ((uintptr_t)p & 15) == 0 && ld % 4 == 0; }
// chunk of eight columns of a token's row in the per-head blocks
__device__ __forceinline__ size_t lb_heads_chunk(int row, int col, int heads, int head_dim, int head_chunks) {
    const int h = col / head_dim, d = col - h * head_dim;
    return ((size_t)(row >> 7) * heads + h) * head_chunks * 2048 + (size_t)((row & 127) >> 3) * head_chunks * 128 + (size_t)(d >> 3) * 128 + (size_t)(row & 7) * 16;
}

__device__ __forceinline__ float lb_warp_sumf(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// two floats in a 64-bit register and their fused multiply-add, one instruction for both
__device__ __forceinline__ uint64_t lb_pack2(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ void lb_unpack2(uint64_t r, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(r)); }
__device__ __forceinline__ uint64_t lb_fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
// sum over all warps of a block; red holds one float per warp, every thread gets the result
__device__ __forceinline__ float lb_block_sumf(float v, float* red) {
    v = lb_warp_sumf(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += red[i];
    return s;
}

__device__ __forceinline__ float lb_sigmoidf(float z) { return __fdiv_rn(1.f, __fadd_rn(1.f, expf(-z))); }
__device__ __forceinline__ float lb_siluf(float z) { return z * lb_sigmoidf(z); }
__device__ __forceinline__ float lb_gelu_erff(float z) { return 0.5f * z * (1.f + erff(z * 0.70710678118654752f)); }
// clamped gated unit of an expert: g = min(gate, limit), u = clamp(up, +-limit), g sigmoid(slope g) (u + 1)
constexpr float kGluSlope = 1.702f;
__device__ __forceinline__ float lb_clamped_glu(float gate, float up, float limit) {
    const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
    return g * lb_sigmoidf(kGluSlope * g) * (u + 1.f);
}
// log of a sigmoid, without overflow for either sign
__device__ __forceinline__ float lb_log_sigmoidf(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// ---- GEMV: one token of each of M <= 8 sequences -------------------------------------------------------------

enum LbDensePro : int {
    LB_DPRO_PLAIN = 0,  // x [M, ldx] as it is
    LB_DPRO_NORM = 1,   // RMS norm with one gain or a weight per column; the normed row may be kept
    LB_DPRO_CONV = 2,   // RMS norm with one gain, then h + causal depthwise convolution of h over time
    LB_DPRO_GATED = 3,  // per-head RMS norm with a weight, times silu or sigmoid of a gate row (output of a recurrent mixer)
    LB_DPRO_MOE = 4,    // routed experts: top-k of the router's logits, RMS norm, times the token's weight for the expert
    LB_DPRO_PAIRS = 5,  // routed experts, second product: one row per (token, choice), summed over the choices
    LB_DPRO_STAGED = 6, // input rows already made by a launch of their own (several tokens; chosen by the launcher)
};
enum LbDenseEpi : int {
    LB_DEPI_F32 = 0,    // out [token, ldo] = acc
    LB_DEPI_RESID = 1,  // out [token, ldo] = res_mult * res + mult * acc
    LB_DEPI_GELU = 2,   // exact gelu (GEMV: float rows, GEMM: image)
    LB_DEPI_GLU = 3,    // clamped gated unit of two products (GEMV: rows of WT per pair, GEMM: image)
    LB_DEPI_IMG = 4,    // GEMM only: image
    LB_DEPI_STAGE = 6,  // GEMV: only the prologue, a CTA per token, into `staged`
    LB_DEPI_SILU = 7,   // silu of the first product times the second (GEMV: float rows, GEMM: image)
    LB_DEPI_HEADS = 5,  // GEMM only: per-head blocks [token block of 128][head][token/8][chunk][token%8][16 B]
};

// What the first expert product leaves for the second: the distinct experts of this pass and, per expert and token, the
// (token, choice) row that goes through it.
constexpr int kMaxLanesPerPass = 8;
constexpr int kMaxTop = 16;
struct LbRouteList {
    int n;
    int expert[kMaxLanesPerPass * kMaxTop];
    int pair[kMaxLanesPerPass * kMaxTop][kMaxLanesPerPass];  // row of token m under this expert, or -1
};

struct LbDenseGemv {
    const uint8_t* w = nullptr;   // image
    const uint8_t* w2 = nullptr;  // GLU, SILU: the second matrix
    size_t group_bytes = 0;       // routed: distance of two experts' images
    int rows = 0, K = 0, slices = 0, M = 0;
    // input
    const float* x = nullptr;
    int ldx = 0;
    const int* row_idx = nullptr;  // token m reads row row_idx[m] of x (null: m)
    const float* gain = nullptr;   // one float, or null: 1
    const float* gain_w = nullptr; // [K], or null: 1
    float* x_out = nullptr;        // NORM: the normed rows [M, ldx], or null
    float eps = 0.f;
    // convolution: weights [taps][ring_ld], ring [lane][taps][ring_ld] of normed inputs (slot = position % taps)
    const float* conv_w = nullptr;
    float* conv_ring = nullptr;
    int taps = 0, ring_ld = 0;
    const int* pos = nullptr;  // position of every token's sequence
    int lane0 = 0;
    // gated heads
    const float* gate = nullptr;  // [M, gate_ld]
    int gate_ld = 0;
    const float* head_w = nullptr;  // [K]
    int head_dim = 0;
    bool gate_sigmoid = false;      // (silu otherwise)
    // routing
    const float* logits = nullptr;  // [M, ldl]
    int ldl = 0, experts = 0, top = 0;
    LbRouteList* list = nullptr;
    const uint8_t* pairs = nullptr;  // [M * top, ldp] rows of WT
    uint4* staged = nullptr;         // [chunk][M rounded up to a power of two] input chunks, set by the launcher
    int ldp = 0;
    // output
    float* out = nullptr;
    uint8_t* out_pairs = nullptr;
    int ldo = 0;
    const float* res = nullptr;  // RESID: [M, ldo], null: out itself
    float mult = 1.f, res_mult = 1.f, limit = 0.f;
};
int lb_dense_gemv(loom_b200_ctx* ctx, int dtype, int pro, int epi, const LbDenseGemv& p);
// tokens of one pass: what the input rows leave room for
int lb_dense_gemv_max_tokens(int K, int dtype);

// ---- GEMM: a block of tokens ---------------------------------------------------------------------------------

struct LbDenseGemm {
    const uint8_t* x = nullptr;  // token image
    const uint8_t* w = nullptr;
    const uint8_t* w2 = nullptr;  // GLU, SILU
    size_t group_bytes = 0;
    int tokens = 0, rows = 0, slices = 0;
    // routed: the rows of x are grouped by expert in whole blocks of 128; *nblocks of them are in use
    const int* nblocks = nullptr;
    const int* block_group = nullptr;
    int max_blocks = 0;
    float* out = nullptr;
    uint8_t* img = nullptr;
    int ldo = 0, img_slices = 0;
    int heads = 0, head_dim = 0, head_chunks = 0;  // per-head blocks: head_dim % 8 == 0, head_chunks 16-byte chunks per row
    float mult = 1.f, res_mult = 1.f, limit = 0.f;  // RESID: out = res_mult * out + mult * acc
    int* status = nullptr;
};
int lb_dense_gemm(loom_b200_ctx* ctx, int dtype, int epi, const LbDenseGemm& p);

template <typename... KArgs, typename... Args>
static inline cudaError_t lb_launch_pdl(loom_b200_ctx* ctx, void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, Args... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid;
    cfg.blockDim = block;
    cfg.dynamicSmemBytes = smem;
    cfg.stream = ctx->stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = ctx->opt_pdl ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kern, KArgs(args)...);
}
#define LB_LAUNCH(ctx, kern, grid, block, smem, ...)                                     \
    do {                                                                                 \
        LB_CUDA((ctx), lb_launch_pdl((ctx), kern, (grid), (block), (smem), __VA_ARGS__)); \
        (ctx)->launches++;                                                               \
    } while (0)
// raises a kernel's shared-memory limit once per process and device (the mask lives with the call site)
#define LB_BIG_SMEM(ctx, kern, bytes)                                                                                        \
    do {                                                                                                                     \
        static std::atomic<unsigned> _done{0};                                                                               \
        if (!(_done.load() & (1u << ((ctx)->device & 31)))) {                                                                \
            LB_CUDA((ctx), cudaFuncSetAttribute((kern), cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(bytes)));         \
            _done.fetch_or(1u << ((ctx)->device & 31));                                                                      \
        }                                                                                                                    \
    } while (0)
