// mixers.cuh -- the steps of a layer stack between its matrix products: norms and the short convolution, gated linear
// attention, the gated delta rule, matrix memories, latent attention, attention over keys and values, routing of tokens to
// experts.  Every mechanism takes its sizes and constants as parameters.
#pragma once
#include "dense.cuh"

// x[n, :] = row tok[n] of a matrix image; ids outside [0, vocab) give a zero row
int lb_embed_image(loom_b200_ctx* ctx, int dtype, const uint8_t* img, int slices, int vocab, int width, const int* tok, int n, float* x, int ldx);
// x[n, :] = gain * rms(table[tok[n], :]); ids outside [0, vocab) give a zero row
int lb_embed_norm(loom_b200_ctx* ctx, int dtype, const void* table, int vocab, int width, const int* tok, int n, const float* gain, float eps,
                  float* x, int ldx);

// RMS norm with one gain or a weight per column of a block of tokens of one sequence, optionally plus a causal depthwise
// convolution of the normed rows over time, written as a token image.  The rows before the block come from the ring (slot =
// position % taps).
struct LbNormBlock {
    const float* x = nullptr;
    int ldx = 0;
    const int* row_idx = nullptr;  // row t of the block is row row_idx[t] of x (null: t)
    int T = 0, width = 0, slices = 0;
    const float* gain = nullptr;    // one float, or null: 1
    const float* gain_w = nullptr;  // [width], or null: 1 (not with a convolution)
    float* rows = nullptr;          // the normed rows [T, ldx], or null; may be x (not with row_idx or a convolution)
    float eps = 0.f;
    const float* conv_w = nullptr;  // [taps][ring_ld], or null: no convolution
    float* ring = nullptr;          // of this sequence: [taps][ring_ld]
    int taps = 1, ring_ld = 0, pos0 = 0;
    uint8_t* img = nullptr;         // or null
};
int lb_norm_block(loom_b200_ctx* ctx, int dtype, const LbNormBlock& p);
// stores the last taps - 1 normed rows of the block in the ring (after lb_norm_block has read it)
int lb_conv_commit(loom_b200_ctx* ctx, const LbNormBlock& p);

// ---- gated linear attention with a decay per key channel ----------------------------------------------------
struct LbGla {
    const float* proj = nullptr;  // [tokens, ldp]: q [heads*dim], k, v [heads*vdim], gate [heads*vdim], decay input [rank]
    int ldp = 0, heads = 0, dim = 0, vdim = 0, rank = 0;
    const float* a2t = nullptr;   // [rank][heads*dim]
    const float* a2b = nullptr;   // [heads*dim]
    float inv_tau = 1.f, qscale = 1.f;
    float* state = nullptr;       // [lane][heads][dim][vdim]
    float* o = nullptr;           // [tokens, ldo]
    int ldo = 0;
};
// Chunks of C tokens of a recurrence S <- (decay) S + k v^T, o = S^T q, once the decays are inside the operands: what a chunk adds,
// the state in front of every chunk, and the outputs.  Scratch of T tokens; lanes of one sequence.
struct LbChunks {
    int C = 0, heads = 0, dim = 0, vdim = 0;
    float *qd = nullptr, *kd = nullptr;  // [T, heads*dim] queries against the state in front of the chunk, keys decayed to the chunk's end
    const float* v = nullptr;            // [T, ldv] values, heads*vdim columns
    int ldv = 0;
    float* decay = nullptr;              // [chunks, heads*dim] decay over a chunk
    float* weights = nullptr;            // [chunks, heads, C, C]
    float* states = nullptr;             // [chunks, heads, dim, vdim]
    float* state = nullptr;              // [heads, dim, vdim] of the sequence
    float* o = nullptr;                  // [T, ldo]
    int ldo = 0;
};
// states[c] = sum over the chunk's tokens of kd v^T
int lb_chunk_states(loom_b200_ctx* ctx, const LbChunks& c, int T);
// states[c] becomes the state in front of chunk c, `state` the one behind the last; fresh: the sequence starts here
int lb_chunk_scan(loom_b200_ctx* ctx, const LbChunks& c, int T, bool fresh);
// o = qd S + weights v
int lb_chunk_out(loom_b200_ctx* ctx, const LbChunks& c, int T);

// one token of each of M sequences
int lb_gla_step(loom_b200_ctx* ctx, const LbGla& p, const int* pos, int lane0, int M);
int lb_gla_chunk(int dim, int rank);
// T tokens of one sequence whose state is `state` (lane 0 of it); qd, kd, decay, weights, states: scratch in chunks of lb_gla_chunk(dim, rank)
int lb_gla_block(loom_b200_ctx* ctx, const LbGla& p, const LbChunks& scratch, int T, int pos0);
// image of (per-head rms of scale * o) * head_w * (silu or sigmoid)(gate); scale [T, heads] or null
int lb_gated_heads_image(loom_b200_ctx* ctx, int dtype, const float* o, int ldo, const float* gate, int ldg, int T, int heads, int vdim, const float* head_w,
                         bool gate_sigmoid, const float* scale, float eps, int slices, uint8_t* img);
// image of plain rows
int lb_rows_image(loom_b200_ctx* ctx, int dtype, const float* x, int ldx, int T, int cols, int slices, uint8_t* img);

// ---- gated delta rule: one decay per head, short convolutions in front -------------------------------------------
struct LbDelta {
    const float* proj = nullptr;  // [tokens, ldp]: q, k [kv_heads*dim], v, gate [heads*vdim], write strength, decay input [heads]
    int ldp = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    const float* conv_w = nullptr;  // [taps][channels], channels = 2*kv_heads*dim + heads*vdim
    float* ring = nullptr;          // [lane][taps][channels] projections in front of the convolution (slot = position % taps)
    int taps = 1;
    const float *a_log = nullptr, *dt_bias = nullptr;  // [heads]
    float qscale = 1.f;
    float* state = nullptr;         // [lane][heads][dim][vdim]
    float* o = nullptr;             // [tokens, ldo]
    int ldo = 0;
};
__host__ __device__ static inline int lb_delta_channels(const LbDelta& p) { return 2 * p.kv_heads * p.dim + p.heads * p.vdim; }
int lb_delta_step(loom_b200_ctx* ctx, const LbDelta& p, const int* pos, int lane0, int M);
int lb_delta_chunk(int dim);
// T tokens of one sequence (state and ring are its own)
struct LbDeltaBlock {
    LbChunks c;                    // qd, kd, weights, states: scratch
    float* qkv = nullptr;          // [T, channels] after convolution, activation and norm
    float *beta = nullptr, *logg = nullptr;  // [T, heads]
    float *wv = nullptr, *wk = nullptr;      // [T, heads*vdim], [T, heads*dim] values and keys after the chunk's own corrections
    float* mix = nullptr;          // [chunks, heads, dim, dim] what a chunk takes out of the state
};
int lb_delta_block(loom_b200_ctx* ctx, const LbDelta& p, const LbDeltaBlock& b, int T, int pos0);

// ---- matrix memory with exponential gates -------------------------------------------------------------------------
struct LbMemory {
    const float* proj = nullptr;  // [tokens, ldp]: q, k [heads*dim], v, gate [heads*vdim], input gate, forget gate [heads]
    int ldp = 0, heads = 0, dim = 0, vdim = 0;
    const float *bias_i = nullptr, *bias_f = nullptr;  // [heads]
    float cap = 1.f, qscale = 1.f;
    float* state = nullptr;       // [lane][heads][dim][vdim], scaled by exp(-m)
    // normaliser and running maximum, twice: a token reads the copy its predecessor wrote (copy = position % 2)
    float* norm = nullptr;        // [lane][2][heads][dim]
    float* top = nullptr;         // [lane][2][heads]
    float* o = nullptr;           // [tokens, ldo]
    int ldo = 0;
};
int lb_memory_step(loom_b200_ctx* ctx, const LbMemory& p, const int* pos, int lane0, int M);
int lb_memory_chunk(int dim);
struct LbMemoryBlock {
    LbChunks c;                   // qd, kd, decay, weights, states: scratch
    float* norms = nullptr;       // [chunks, heads, dim] what a chunk adds to the normaliser, then the normaliser in front of it
    float* sums = nullptr;        // [T, heads] sums of a token's weights inside its chunk
    float* tops = nullptr;        // [T, heads] running maximum
    float *gate_i = nullptr, *gate_f = nullptr;  // [heads, T] log gates
    float* scale = nullptr;       // [T, heads] out: what the outputs still have to be multiplied by
};
// T tokens of one sequence (state, norm and top are its own)
int lb_memory_block(loom_b200_ctx* ctx, const LbMemory& p, const LbMemoryBlock& b, int T, int pos0);

// ---- softmax attention over cached keys and values ------------------------------------------------------------------
//
// Keys are kept per head in blocks of 128 positions [block][kv head][position/8][chunk][position%8][16 B], values transposed in an
// image of [kv_heads * vdim rounded up to 8] x positions, both as rings of `ring` positions (a multiple of 128; position p is row
// p % ring).  With chunks of c positions a ring only has to hold a chunk and a block of tokens.
constexpr int kBiasFront = 192, kBiasBack = 64;  // entries in front of distance 0 and behind the last one of a bias row
struct LbAttention {
    const float* proj = nullptr;  // [tokens, ldp]: q [heads*dim], k [kv_heads*dim], v [kv_heads*vdim], gate [heads] (with head_gate)
    int ldp = 0, heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    float scale = 1.f, eps = 0.f;
    bool qk_norm = false, sink = false, head_gate = false;
    int chunk = 0;                // 0: every earlier position is visible
    const float *bias = nullptr, *bias_log2 = nullptr;  // [heads][bias_ld], entry kBiasFront + distance; the second times log2(e)
    int bias_len = 0, bias_ld = 0;  // distances from bias_len - 1 on share the last value
    uint8_t *k = nullptr, *vt = nullptr;  // [lane] caches
    size_t k_lane = 0, vt_lane = 0;
    int ring = 0, slices = 0;     // slices: K slices of a row of vt
    bool mma = false;             // the step runs on the tensor cores (lb_attention_step_mma)
    const int* pos = nullptr;     // position of every token (one token per sequence), or null: token t is at pos0 + t of lane0
    int pos0 = 0, lane0 = 0;
};
bool lb_attention_step_mma(int dim, int vdim, int dtype);
int lb_attention_kchunks(int dim, int dtype);
size_t lb_attention_k_bytes(int kv_heads, int dim, int ring, int dtype);
size_t lb_attention_vt_bytes(int kv_heads, int vdim, int ring, int dtype);
// keys and values of a block into the cache and, bf16 with q_img, its queries into per-head blocks (lb_attention_q_bytes)
size_t lb_attention_q_bytes(const LbAttention& p, int rows);
int lb_attention_store(loom_b200_ctx* ctx, int dtype, const LbAttention& p, int T, uint8_t* q_img);
// one token of each sequence (stores its key and value too), or, with pos null, tokens whose keys and values are stored.
// part: lb_attention_part_elems floats; count: lb_attention_counters zeroed integers, zero again afterwards
int lb_attention_splits(loom_b200_ctx* ctx, const LbAttention& p, int tokens);
size_t lb_attention_part_elems(loom_b200_ctx* ctx, const LbAttention& p, int tokens);
size_t lb_attention_counters(const LbAttention& p, int tokens);
int lb_attention_step(loom_b200_ctx* ctx, int dtype, const LbAttention& p, int tokens, float* part, unsigned* count, float* out, int ldo);
// bf16, a block of stored tokens on the tensor cores; out: token image of heads*vdim columns
bool lb_attention_block_supported(const LbAttention& p);
int lb_attention_block(loom_b200_ctx* ctx, const LbAttention& p, int T, const uint8_t* q_img, uint8_t* out, int out_slices);

// The tensor-core kernel under it (and under latent attention): 128 query tokens x one head per CTA, tiles of 64 positions.
struct LbAttnBlock {
    const uint8_t* q = nullptr;   // [token block of 128][head][row/8][chunk][row%8][16 B]
    const uint8_t* k = nullptr;   // the same of positions and kv heads
    const uint8_t* vt = nullptr;  // image of [kv_heads*vrows] x positions
    int heads = 0, kv_heads = 0, dchunks = 0, vdim = 0, vrows = 0, vslices = 0;  // dchunks: 16-byte chunks of a query row (even); vrows: rows of a head in vt (a multiple of 8)
    int T = 0, pos0 = 0;
    float scale_log2 = 0.f;       // factor of the scores times log2(e) (not negative without `general`)
    uint8_t* out = nullptr;       // token image of heads*vdim columns
    int out_slices = 0;
    // general: any of chunks, distance bias, sink, gate, ring of positions
    bool general = false;
    int chunk = 0, ring = 0;
    const float* bias = nullptr;  // log2(e) times the bias, rows of bias_ld as in LbAttention; or null
    int bias_len = 0, bias_ld = 0;
    bool sink = false;
    const float* gate = nullptr;  // [T, ldg], one number per head before the sigmoid, or null
    int ldg = 0;
    int* status = nullptr;
};
int lb_attn_block(loom_b200_ctx* ctx, const LbAttnBlock& p);

// ---- latent attention ------------------------------------------------------------------------------------------
struct LbLatent {
    const float* q = nullptr;      // [tokens, ldq]: heads*dim queries
    int ldq = 0, heads = 0, dim = 0, vdim = 0, rank = 0;
    float scale = 1.f;
    const uint8_t *uk = nullptr, *uv = nullptr;  // images of [heads*dim, rank] and [heads*vdim, rank]
    int slices = 0;                // K slices of rank
    uint8_t* cache = nullptr;      // [lane] images of positions x rank
    size_t lane_bytes = 0;
    const int* pos = nullptr;      // position of every token (one token per sequence), or null: token t is at pos0 + t of lane0
    int pos0 = 0, lane0 = 0, max_seq = 0;
};
// latent rows: rms of raw * weight into the cache
int lb_latent_store(loom_b200_ctx* ctx, int dtype, const LbLatent& p, const float* raw, int ldr, const float* weight, float eps, int tokens);
// queries in latent space: ql[token, head, rank] = scale * W_uk[head]^T q; with raw, the tokens' latents are stored by the same launch
int lb_latent_absorb_q(loom_b200_ctx* ctx, int dtype, const LbLatent& p, const float* raw, int ldr, const float* weight, float eps, int tokens, float* ql);
// attention over the latents: ol[token, head, rank] = sum_j softmax_j(ql . c_j) c_j
int lb_latent_attention(loom_b200_ctx* ctx, int dtype, const LbLatent& p, int tokens, const float* ql, float* ol);
// out[token, heads*vdim] = W_uv[head] ol
int lb_latent_absorb_v(loom_b200_ctx* ctx, int dtype, const LbLatent& p, int tokens, const float* ol, float* out, int ldo);

// bf16, one token per sequence or a few tokens of one: every latent is read once for up to sixteen heads, the positions split over
// `splits` CTAs whose results meet in front of the value rows.  part: [tokens, heads, splits, rank + 2]
bool lb_latent_step_supported(const LbLatent& p);
int lb_latent_step_splits(loom_b200_ctx* ctx, const LbLatent& p, int tokens);
int lb_latent_step(loom_b200_ctx* ctx, const LbLatent& p, int tokens, const float* ql, float* part, int splits, float* out, int ldo);
// bf16, a block of tokens on the tensor cores: keys and values of every position are expanded from the latents.  q_img and k_img hold
// lb_latent_heads_bytes of T and pos0 + T rows, vt_img is an image of [heads*vdim] x positions (vt_slices K slices); the pads of
// all three are zero.  out: token image of heads*vdim columns
bool lb_latent_block_supported(const LbLatent& p);
size_t lb_latent_heads_bytes(const LbLatent& p, int rows);
int lb_latent_block(loom_b200_ctx* ctx, const LbLatent& p, int T, uint8_t* q_img, uint8_t* k_img, uint8_t* vt_img, int vt_slices, uint8_t* out,
                    int out_slices);

// ---- routing of a token block ------------------------------------------------------------------------------------
struct LbRouteBlock {
    int T = 0, experts = 0, top = 0;
    const float* logits = nullptr;  // [T, ldl]
    int ldl = 0;
    int* idx = nullptr;     // [T, top] chosen experts
    float* score = nullptr; // [T, top]
    int* slot = nullptr;    // [T, top] rank of the pair among its expert's pairs, then its row of the grouped image
    int* count = nullptr;   // [experts]
    int* offset = nullptr;  // [experts] first row
    int* block_group = nullptr;  // expert of every 128-row block
    int* nblocks = nullptr;
};
static inline int lb_route_max_blocks(int T, int experts, int top) {
    // every used expert wastes less than one block
    const int pairs = T * top;
    return pairs / kImgRows + (experts < pairs ? experts : pairs);
}
// chooses the experts of every token and lays the pairs out by expert in whole 128-row blocks
int lb_route_block(loom_b200_ctx* ctx, const LbRouteBlock& p);
// grouped image: row of pair (t, j) = score * gain * rms(x[t])
int lb_route_gather(loom_b200_ctx* ctx, int dtype, const LbRouteBlock& p, const float* x, int ldx, int width, const float* gain, float eps, int slices,
                    uint8_t* img);
// x[t] += mult * sum_j y[row of (t, j)]
int lb_route_combine(loom_b200_ctx* ctx, const LbRouteBlock& p, const float* y, int ldy, float mult, int width, float* x, int ldx);
