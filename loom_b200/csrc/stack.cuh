// stack.cuh -- a decoder whose layers are given one by one (mixer + feed-forward), driven by the decoder loop in decoder.cu:
// the loop owns positions, current tokens, output rings, logits rows and the recorded step; the stack owns the layers, the
// per-sequence mixer states and the scratch of a pass.
#pragma once
#include <vector>

#include "mixers.cuh"

struct LbLayer {
    loom_b200_layer_spec s{};
    loom_b200_layer_weights w{};  // matrices borrowed
    bool ready = false;
    // device copies of the small vectors
    float* scal = nullptr;        // norm1, norm2
    float *norm1_w = nullptr, *norm2_w = nullptr;  // weights per column, or null
    float* mixer_norm = nullptr;  // latent: [rank]; recurrent mixers: [heads*vdim]
    float *decay_wt = nullptr, *decay_b = nullptr, *conv_w = nullptr;
    float *bias = nullptr, *bias_log2 = nullptr;   // attention: bias by distance
    int bias_len = 0, bias_ld = 0;
    float *a_log = nullptr, *dt_bias = nullptr;    // delta rule
    float *gate_b_i = nullptr, *gate_b_f = nullptr;  // matrix memory
    // state of every sequence
    float* conv_ring = nullptr;   // [lane][taps][ring_ld]; delta rule: [lane][conv][channels]
    float* state = nullptr;       // recurrent mixers: [lane][heads][dim][vdim]
    float *mem_norm = nullptr, *mem_top = nullptr;   // matrix memory: [lane][2][heads][dim], [lane][2][heads]
    uint8_t *k_cache = nullptr, *vt_cache = nullptr;  // attention
    size_t k_lane = 0, vt_lane = 0;
    int ring = 0;
    uint8_t* latent = nullptr;    // [lane] image of positions x rank
    size_t latent_lane = 0;
    int in_cols = 0;              // rows of w.in
};

struct LbStack {
    loom_b200_stack_dims d{};
    int ldx = 0;                  // floats of a residual row
    std::vector<LbLayer> layers;
    int lanes = 1;
    const void* table = nullptr;  // embedding rows in the stack's dtype (borrowed)
    const loom_b200_matrix* head = nullptr;  // also the embedding without a table
    float* scal = nullptr;        // embedding norm, final norm
    float* final_w = nullptr;     // weights of the final norm, or null
    // scratch of a pass of up to eight sequences
    float* y = nullptr;           // norms after the sum: the sum that waits for its norm (x is the normed row)
    float *x = nullptr, *proj = nullptr, *o = nullptr, *mid = nullptr, *ql = nullptr, *ol = nullptr, *rlog = nullptr;
    uint8_t* pairs = nullptr;
    LbRouteList* list = nullptr;
    float* attn_part = nullptr;
    unsigned* attn_count = nullptr;  // zero between launches
    int ldp = 0, ldo = 0, ldm = 0, lde = 0, ldr = 0;
    bool scratch_ready = false;
    // scratch of a token block
    int cap = 0;
    int* pf_tok = nullptr;
    float *pf_x = nullptr, *pf_proj = nullptr, *pf_o = nullptr, *pf_part = nullptr, *pf_ql = nullptr,
          *pf_ol = nullptr, *pf_y = nullptr, *pf_rlog = nullptr, *pf_score = nullptr, *pf_logits = nullptr;
    uint8_t *pf_h = nullptr, *pf_io = nullptr, *pf_act = nullptr, *pf_gx = nullptr, *pf_ga = nullptr;
    uint8_t* pf_mix = nullptr;    // scratch of a recurrent mixer (mixer_scratch in stack.cu)
    uint8_t *pf_qi = nullptr, *pf_k = nullptr, *pf_v = nullptr;
    size_t kv_rows = 0;
    int *pf_idx = nullptr, *pf_slot = nullptr, *pf_count = nullptr, *pf_offset = nullptr, *pf_bg = nullptr, *pf_nb = nullptr, *pf_rows = nullptr;
    int ldl = 0;                  // floats of a row of pf_logits
};

constexpr int kStackBlock = 2048;     // tokens per pass of a prompt
constexpr int kStackHeadRows = 128;   // logits rows per pass of the head

void lb_stack_free(LbStack* st);
// checks and installs a layer and allocates its state for `lanes` sequences
int lb_stack_set_layer(loom_b200_ctx* ctx, LbStack* st, int layer, const loom_b200_layer_spec& spec, const loom_b200_layer_weights& weights, int lanes);
// tokens of one pass over several sequences
int lb_stack_max_lanes(const LbStack* st);
int lb_stack_ready(loom_b200_ctx* ctx, LbStack* st);
// one token of each of sequences lane0 .. lane0 + M - 1 (tok[m], position pos[m]) through every layer; the residual rows stay in st->x
int lb_stack_step(loom_b200_ctx* ctx, LbStack* st, const int* tok, const int* pos, int lane0, int M);
// T tokens of one sequence at positions pos0 .. through every layer (ids in st->pf_tok); residual rows in st->pf_x
int lb_stack_block(loom_b200_ctx* ctx, LbStack* st, int T, int pos0, int lane);
int lb_stack_ensure_block(loom_b200_ctx* ctx, LbStack* st, int tokens);
// logits of n rows of x: row rows_dev[i] (null: i) -> out + i * ldo; up to eight
int lb_stack_head(loom_b200_ctx* ctx, LbStack* st, const float* x, const int* rows_dev, int n, float* out, int ldo);
// logits of up to kStackHeadRows rows of pf_x (indices in st->pf_rows) into st->pf_logits
int lb_stack_head_block(loom_b200_ctx* ctx, LbStack* st, int n);
