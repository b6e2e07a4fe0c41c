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
    float *mixer_norm = nullptr, *decay_wt = nullptr, *decay_b = nullptr, *conv_w = nullptr;
    // state of every sequence
    float* conv_ring = nullptr;   // [lane][taps][ring_ld]
    float* gla_state = nullptr;   // [lane][heads][dim][vdim]
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
    const loom_b200_matrix* head = nullptr;
    float* scal = nullptr;        // embedding norm, final norm
    // scratch of a pass of up to eight sequences
    float *x = nullptr, *proj = nullptr, *o = nullptr, *mid = nullptr, *ql = nullptr, *ol = nullptr, *rlog = nullptr;
    uint8_t* pairs = nullptr;
    LbRouteList* list = nullptr;
    float* attn_part = nullptr;
    int ldp = 0, ldo = 0, ldm = 0, lde = 0, ldr = 0;
    bool scratch_ready = false;
    // scratch of a token block
    int cap = 0;
    int* pf_tok = nullptr;
    float *pf_x = nullptr, *pf_proj = nullptr, *pf_o = nullptr, *pf_qd = nullptr, *pf_kd = nullptr, *pf_cw = nullptr, *pf_part = nullptr, *pf_cs = nullptr, *pf_cd = nullptr, *pf_ql = nullptr,
          *pf_ol = nullptr, *pf_y = nullptr, *pf_rlog = nullptr, *pf_score = nullptr, *pf_logits = nullptr;
    uint8_t *pf_h = nullptr, *pf_io = nullptr, *pf_act = nullptr, *pf_gx = nullptr, *pf_ga = nullptr;
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
