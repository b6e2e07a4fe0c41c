// mixers.cuh -- the steps of a layer stack between its matrix products: norms and the short convolution, gated linear
// attention, latent attention, routing of tokens to experts.  Every mechanism takes its sizes and constants as parameters.
#pragma once
#include "dense.cuh"

// x[n, :] = gain * rms(table[tok[n], :]); ids outside [0, vocab) give a zero row
int lb_embed_norm(loom_b200_ctx* ctx, int dtype, const void* table, int vocab, int width, const int* tok, int n, const float* gain, float eps,
                  float* x, int ldx);

// RMS norm with one gain of a block of tokens of one sequence, optionally plus a causal depthwise convolution of the normed
// rows over time, written as a token image.  The rows before the block come from the ring (slot = position % taps).
struct LbNormBlock {
    const float* x = nullptr;
    int ldx = 0;
    const int* row_idx = nullptr;  // row t of the block is row row_idx[t] of x (null: t)
    int T = 0, width = 0, slices = 0;
    const float* gain = nullptr;
    float eps = 0.f;
    const float* conv_w = nullptr;  // [taps][ring_ld], or null: no convolution
    float* ring = nullptr;          // of this sequence: [taps][ring_ld]
    int taps = 1, ring_ld = 0, pos0 = 0;
    uint8_t* img = nullptr;
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
// one token of each of M sequences
int lb_gla_step(loom_b200_ctx* ctx, const LbGla& p, const int* pos, int lane0, int M);
// scratch of a block of T tokens in chunks of C = lb_gla_chunk(dim, rank)
struct LbGlaBlock {
    int C = 0;
    float *qd = nullptr, *kd = nullptr;  // [T, heads*dim] queries decayed from the chunk's start, keys decayed to its end
    float* decay = nullptr;              // [chunks, heads*dim] decay over a chunk
    float* weights = nullptr;            // [chunks, heads, C, C]
    float* states = nullptr;             // [chunks, heads, dim, vdim]
};
int lb_gla_chunk(int dim, int rank);
// T tokens of one sequence whose state is `state` (lane 0 of it)
int lb_gla_block(loom_b200_ctx* ctx, const LbGla& p, const LbGlaBlock& b, int T, int pos0);
// image of (per-head rms of o) * head_w * silu(gate)
int lb_gated_heads_image(loom_b200_ctx* ctx, int dtype, const float* o, int ldo, const float* gate, int ldg, int T, int heads, int vdim, const float* head_w,
                         float eps, int slices, uint8_t* img);
// image of plain rows
int lb_rows_image(loom_b200_ctx* ctx, int dtype, const float* x, int ldx, int T, int cols, int slices, uint8_t* img);

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
