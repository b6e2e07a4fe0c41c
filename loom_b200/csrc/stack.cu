// stack.cu -- the layers of a stack decoder: weights and states per layer, the one-token-per-sequence step and the token block.
//
// Step, per layer (M <= 8 sequences, one token each; every launch chained by programmatic dependent launch):
//   gated linear attention   {norm + short convolution + input projections} -> {decay, state update, read-out}
//                            -> {per-head norm, gate, output projection, residual}
//   latent attention         {norm + short convolution + query / latent projections} -> {queries into latent space, latent
//                            norm, cache} -> {attention over the latents} -> {values} -> {output projection, residual}
//   attention                {norm + q / k / v / gate projections} -> {head norms, cache, attention, head gate} -> {output projection,
//                            residual}
//   delta rule, matrix memory  {norm + projections} -> {convolutions / gates, state update, read-out} -> {per-head norm, gate, output
//                            projection, residual}
//   feed-forward             dense {norm, up, gelu} -> {down, residual}; gated {norm, gate / up, product} -> {down, residual}; routed
//                            {norm, router} -> {choice, norm, gate / up, clamped unit} -> {down of every chosen expert, sum, residual}
//
// Norms after the sum: the residual products write the sum, the next product's prologue norms it and keeps the normed row, which is
// what the next sum adds to.
#include "stack.cuh"

#include <algorithm>
#include <cmath>

namespace {

bool is_bf16(const LbStack* st) { return st->d.dtype == LOOM_B200_DTYPE_BF16; }

int hv_of(const loom_b200_layer_spec& s) { return s.heads * s.vdim; }

LbGla gla_of(const LbLayer& l, const float* proj, int ldp, float* o, int ldo, int lane) {
    LbGla g;
    const loom_b200_layer_spec& s = l.s;
    g.proj = proj;
    g.ldp = ldp;
    g.heads = s.heads;
    g.dim = s.dim;
    g.vdim = s.vdim;
    g.rank = s.rank;
    g.a2t = l.decay_wt;
    g.a2b = l.decay_b;
    g.inv_tau = (float)(1.0 / s.tau);
    g.qscale = (float)(1.0 / std::sqrt((double)s.dim));
    g.state = l.state + (size_t)lane * s.heads * s.dim * s.vdim;
    g.o = o;
    g.ldo = ldo;
    return g;
}

LbDelta delta_of(const LbLayer& l, const float* proj, int ldp, float* o, int ldo, int lane) {
    LbDelta p;
    const loom_b200_layer_spec& s = l.s;
    p.proj = proj;
    p.ldp = ldp;
    p.heads = s.heads;
    p.kv_heads = s.kv_heads;
    p.dim = s.dim;
    p.vdim = s.vdim;
    p.conv_w = l.conv_w;
    p.taps = s.conv;
    p.ring = l.conv_ring + (size_t)lane * s.conv * lb_delta_channels(p);
    p.a_log = l.a_log;
    p.dt_bias = l.dt_bias;
    p.qscale = (float)(1.0 / std::sqrt((double)s.dim));
    p.state = l.state + (size_t)lane * s.heads * s.dim * s.vdim;
    p.o = o;
    p.ldo = ldo;
    return p;
}

LbMemory memory_of(const LbLayer& l, const float* proj, int ldp, float* o, int ldo, int lane) {
    LbMemory p;
    const loom_b200_layer_spec& s = l.s;
    p.proj = proj;
    p.ldp = ldp;
    p.heads = s.heads;
    p.dim = s.dim;
    p.vdim = s.vdim;
    p.bias_i = l.gate_b_i;
    p.bias_f = l.gate_b_f;
    p.cap = (float)s.gate_cap;
    p.qscale = (float)(1.0 / std::sqrt((double)s.dim));
    p.state = l.state + (size_t)lane * s.heads * s.dim * s.vdim;
    p.norm = l.mem_norm + (size_t)lane * 2 * s.heads * s.dim;
    p.top = l.mem_top + (size_t)lane * 2 * s.heads;
    p.o = o;
    p.ldo = ldo;
    return p;
}

LbAttention attention_of(const LbStack* st, const LbLayer& l, const float* proj, int ldp) {
    LbAttention p;
    const loom_b200_layer_spec& s = l.s;
    p.proj = proj;
    p.ldp = ldp;
    p.heads = s.heads;
    p.kv_heads = s.kv_heads;
    p.dim = s.dim;
    p.vdim = s.vdim;
    p.scale = (float)s.scale;
    p.eps = (float)st->d.norm_eps;
    p.qk_norm = s.qk_norm != 0;
    p.sink = s.sink != 0;
    p.head_gate = s.head_gate != 0;
    p.chunk = s.chunk;
    p.bias = l.bias;
    p.bias_log2 = l.bias_log2;
    p.bias_len = l.bias_len;
    p.bias_ld = l.bias_ld;
    p.k = l.k_cache;
    p.vt = l.vt_cache;
    p.k_lane = l.k_lane;
    p.vt_lane = l.vt_lane;
    p.ring = l.ring;
    p.slices = lb_slices_of(l.ring, st->d.dtype);
    p.mma = lb_attention_step_mma(s.dim, s.vdim, st->d.dtype);
    return p;
}

// Scratch of a recurrent mixer for a block of T tokens, carved out of `base` (null: only counted).  Returns its bytes.
struct MixerScratch {
    LbChunks c;
    LbDeltaBlock delta;
    LbMemoryBlock mem;
};
size_t mixer_scratch(const LbLayer& l, int T, uint8_t* base, MixerScratch& m) {
    const loom_b200_layer_spec& s = l.s;
    size_t at = 0;
    auto take = [&](float*& p, size_t n) {
        p = base ? reinterpret_cast<float*>(base + at) : nullptr;
        at += (n * sizeof(float) + 255) / 256 * 256;
    };
    const size_t H = s.heads, D = s.dim, V = s.vdim, t = T;
    size_t C = 0;
    if (s.mixer == LOOM_B200_MIXER_GLA) C = lb_gla_chunk(s.dim, s.rank);
    if (s.mixer == LOOM_B200_MIXER_DELTA) C = lb_delta_chunk(s.dim);
    if (s.mixer == LOOM_B200_MIXER_MLSTM) C = lb_memory_chunk(s.dim);
    if (C == 0) return 0;
    const size_t n = lb_ceil_div(T, (int)C);
    take(m.c.qd, t * H * D);
    take(m.c.kd, t * H * D);
    take(m.c.decay, n * H * D);
    take(m.c.weights, n * H * C * C);
    take(m.c.states, n * H * D * V);
    if (s.mixer == LOOM_B200_MIXER_DELTA) {
        take(m.delta.qkv, t * (2 * s.kv_heads * D + H * V));
        take(m.delta.beta, t * H);
        take(m.delta.logg, t * H);
        take(m.delta.wv, t * H * V);
        take(m.delta.wk, t * H * D);
        take(m.delta.mix, n * H * D * D);
    }
    if (s.mixer == LOOM_B200_MIXER_MLSTM) {
        take(m.mem.norms, n * H * D);
        take(m.mem.sums, t * H);
        take(m.mem.tops, t * H);
        take(m.mem.scale, t * H);
        take(m.mem.gate_i, t * H);
        take(m.mem.gate_f, t * H);
    }
    m.delta.c = m.mem.c = m.c;
    return at;
}

// The distance bias of every head by distance, with the last value repeated behind it and zeros in front: half of the buckets hold
// one distance each, the others grow in equal ratios up to bias_max.
int put_bias(loom_b200_ctx* ctx, LbLayer& l, const float* rel) {
    const loom_b200_layer_spec& s = l.s;
    const int B = s.buckets, near = B / 2;
    auto bucket = [&](int n) {
        if (n < near) return n;
        const double x = std::log((double)n / near) / std::log(s.bias_max / near) * (B - near);
        return x >= B - 1 - near ? B - 1 : near + (int)std::floor(x);
    };
    int len = near;
    while (len < (1 << 24) && bucket(len) < B - 1) ++len;
    ++len;
    l.bias_len = len;
    l.bias_ld = lb_round_up(kBiasFront + len + kBiasBack, 4);
    std::vector<float> t((size_t)s.heads * l.bias_ld, 0.f), u;
    for (int h = 0; h < s.heads; ++h)
        for (int i = kBiasFront; i < l.bias_ld; ++i) t[(size_t)h * l.bias_ld + i] = rel[(size_t)bucket(std::min(i - kBiasFront, len - 1)) * s.heads + h];
    u = t;
    for (auto& x : u) x = (float)((double)x * 1.4426950408889634);
    LB_CUDA(ctx, cudaMalloc((void**)&l.bias, t.size() * 4));
    LB_CUDA(ctx, cudaMalloc((void**)&l.bias_log2, t.size() * 4));
    LB_CUDA(ctx, cudaMemcpyAsync(l.bias, t.data(), t.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
    LB_CUDA(ctx, cudaMemcpyAsync(l.bias_log2, u.data(), u.size() * 4, cudaMemcpyHostToDevice, ctx->stream));
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    return 0;
}

LbLatent latent_of(const LbStack* st, const LbLayer& l, const float* proj, int ldp) {
    const LbLayer& src = l.s.kv_from >= 0 ? st->layers[l.s.kv_from] : l;
    LbLatent p;
    p.q = proj;
    p.ldq = ldp;
    p.heads = l.s.heads;
    p.dim = l.s.dim;
    p.vdim = l.s.vdim;
    p.rank = l.s.rank;
    p.scale = (float)l.s.scale;
    p.uk = l.w.up_k->data;
    p.uv = l.w.up_v->data;
    p.slices = l.w.up_k->slices;
    p.cache = src.latent;
    p.lane_bytes = src.latent_lane;
    p.max_seq = st->d.max_seq_len;
    return p;
}

constexpr int kAttentionStepTokens = 8;  // tokens of a portion that go through the attention step's kernel
constexpr int kLatentStepTokens = 32;  // tokens of a portion that go through the step's attention kernels

// attention of a few tokens in latent space, values applied: out [tokens, ldo].  raw: the latent projections that go into the cache
// first (row stride of the queries), or null
int latent_few(loom_b200_ctx* ctx, LbStack* st, int dt, const LbLatent& a, const float* raw, const float* norm, int tokens, float* ql, float* ol, float* part,
               float* out, int ldo) {
    if (int rc = lb_latent_absorb_q(ctx, dt, a, raw, a.ldq, norm, (float)st->d.norm_eps, tokens, ql)) return rc;
    if (dt == LOOM_B200_DTYPE_BF16 && lb_latent_step_supported(a))
        return lb_latent_step(ctx, a, tokens, ql, part, lb_latent_step_splits(ctx, a, tokens), out, ldo);
    if (int rc = lb_latent_attention(ctx, dt, a, tokens, ql, ol)) return rc;
    return lb_latent_absorb_v(ctx, dt, a, tokens, ol, out, ldo);
}

// tokens of a block of T that an attention layer sends through the step's kernel
int attention_step_tokens(const LbStack* st, const LbLayer& l, int T) {
    const bool tc = is_bf16(st) && lb_attention_block_supported(attention_of(st, l, nullptr, 0));
    return tc ? std::min(T, kAttentionStepTokens) : T;
}

// floats of the split results of up to `tokens` tokens of any layer
size_t attn_part_elems(loom_b200_ctx* ctx, LbStack* st, int tokens) {
    size_t n = 0;
    for (auto& l : st->layers) {
        if (l.s.mixer == LOOM_B200_MIXER_ATTENTION) {
            const LbAttention a = attention_of(st, l, nullptr, 0);
            for (int t = 1, most = attention_step_tokens(st, l, tokens); t <= most; ++t)
                if (lb_attention_splits(ctx, a, t) > 1) n = std::max(n, lb_attention_part_elems(ctx, a, t));
        }
        if (l.s.mixer != LOOM_B200_MIXER_LATENT || !is_bf16(st)) continue;
        const LbLatent a = latent_of(st, l, nullptr, 0);
        for (int t = 1; t <= std::min(tokens, kLatentStepTokens); ++t) n = std::max(n, (size_t)t * l.s.heads * lb_latent_step_splits(ctx, a, t) * (l.s.rank + 2));
    }
    return n;
}

// keys and transposed values of `rows` positions, expanded from the latents for a block
int ensure_kv(loom_b200_ctx* ctx, LbStack* st, int rows) {
    if ((size_t)rows <= st->kv_rows) return 0;
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "stack scratch would grow while recording a graph");
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    if (st->pf_k) cudaFree(st->pf_k);
    if (st->pf_v) cudaFree(st->pf_v);
    st->pf_k = st->pf_v = nullptr;
    st->kv_rows = 0;
    const int n = lb_round_up(std::min(std::max(2 * rows, 1024), std::max(rows, st->d.max_seq_len)), kImgRows);
    size_t k = 0, v = 0;
    for (auto& l : st->layers) {
        if (l.s.mixer != LOOM_B200_MIXER_LATENT) continue;
        const LbLatent a = latent_of(st, l, nullptr, 0);
        k = std::max(k, lb_latent_heads_bytes(a, n));
        v = std::max(v, lb_img_bytes(hv_of(l.s), n, LOOM_B200_DTYPE_BF16));
    }
    LB_CUDA(ctx, cudaMalloc(&st->pf_k, k));
    LB_CUDA(ctx, cudaMalloc(&st->pf_v, v));
    LB_CUDA(ctx, cudaMemsetAsync(st->pf_k, 0, k, ctx->stream));
    LB_CUDA(ctx, cudaMemsetAsync(st->pf_v, 0, v, ctx->stream));
    st->kv_rows = n;
    return 0;
}

int ensure_step_scratch(loom_b200_ctx* ctx, LbStack* st) {
    if (st->scratch_ready) return 0;
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "stack scratch would be allocated while recording a graph");
    const int M = kMaxLanesPerPass;
    int in_cols = 0, hv = 0, ff = 0, eff = 0, top = 0, experts = 0, hr = 0;
    size_t counters = 0;
    for (auto& l : st->layers) {
        in_cols = std::max(in_cols, l.in_cols);
        hv = std::max(hv, hv_of(l.s));
        if (l.s.mixer == LOOM_B200_MIXER_LATENT) hr = std::max(hr, l.s.heads * l.s.rank);
        if (l.s.mixer == LOOM_B200_MIXER_ATTENTION)  // a block's tokens count too: kStackBlock of them at most
            counters = std::max(counters, lb_attention_counters(attention_of(st, l, nullptr, 0), std::max(M, attention_step_tokens(st, l, kStackBlock))));
        if (l.s.ffn == LOOM_B200_FFN_DENSE || l.s.ffn == LOOM_B200_FFN_GATED) ff = std::max(ff, l.s.ff);
        if (l.s.ffn == LOOM_B200_FFN_MOE) {
            eff = std::max(eff, l.w.down->slices * lb_slice_cols(st->d.dtype));
            top = std::max(top, l.s.top);
            experts = std::max(experts, l.s.experts);
        }
    }
    st->ldp = lb_round_up(in_cols, 8);
    st->ldo = lb_round_up(hv, 8);
    st->ldm = lb_round_up(ff, 8);
    st->lde = eff;
    st->ldr = lb_round_up(experts, 8);
    auto A = [&](auto** p, size_t bytes) -> int {
        if (bytes == 0) return 0;
        LB_CUDA(ctx, cudaMalloc((void**)p, bytes));
        LB_CUDA(ctx, cudaMemsetAsync(*p, 0, bytes, ctx->stream));
        return 0;
    };
    if (int rc = A(&st->x, (size_t)M * st->ldx * 4)) return rc;
    if (st->d.post_norm)
        if (int rc = A(&st->y, (size_t)M * st->ldx * 4)) return rc;
    if (int rc = A(&st->proj, (size_t)M * st->ldp * 4)) return rc;
    if (int rc = A(&st->o, (size_t)M * st->ldo * 4)) return rc;
    if (int rc = A(&st->mid, (size_t)M * st->ldm * 4)) return rc;
    if (int rc = A(&st->ql, (size_t)M * hr * 4)) return rc;
    if (int rc = A(&st->ol, (size_t)M * hr * 4)) return rc;
    if (int rc = A(&st->rlog, (size_t)M * st->ldr * 4)) return rc;
    if (int rc = A(&st->attn_part, attn_part_elems(ctx, st, M) * 4)) return rc;
    if (int rc = A(&st->attn_count, counters * 4)) return rc;
    if (int rc = A(&st->pairs, (size_t)M * top * eff * (is_bf16(st) ? 2 : 4))) return rc;
    if (int rc = A(&st->list, sizeof(LbRouteList))) return rc;
    st->scratch_ready = true;
    return 0;
}

bool recurrent(const loom_b200_layer_spec& s) {
    return s.mixer == LOOM_B200_MIXER_GLA || s.mixer == LOOM_B200_MIXER_DELTA || s.mixer == LOOM_B200_MIXER_MLSTM;
}

// first column of a recurrent mixer's gate row in the projections: behind q, k and v
int gate_col(const loom_b200_layer_spec& s) { return 2 * (s.mixer == LOOM_B200_MIXER_DELTA ? s.kv_heads : s.heads) * s.dim + hv_of(s); }

int embed(loom_b200_ctx* ctx, LbStack* st, const int* tok, int n, float* x) {
    const loom_b200_stack_dims& d = st->d;
    if (!st->table) return lb_embed_image(ctx, d.dtype, st->head->data, st->head->slices, d.vocab, d.width, tok, n, x, st->ldx);
    return lb_embed_norm(ctx, d.dtype, st->table, d.vocab, d.width, tok, n, st->scal, (float)d.norm_eps, x, st->ldx);
}

void free_block(LbStack* st) {
    void* ptrs[] = {st->pf_tok, st->pf_x, st->pf_proj, st->pf_o, st->pf_mix, st->pf_part, st->pf_ql, st->pf_ol, st->pf_y, st->pf_rlog,
                    st->pf_score, st->pf_logits, st->pf_h, st->pf_io, st->pf_act, st->pf_gx, st->pf_ga, st->pf_idx, st->pf_slot, st->pf_count,
                    st->pf_offset, st->pf_bg, st->pf_nb, st->pf_rows, st->pf_qi, st->pf_k, st->pf_v};
    for (void* p : ptrs)
        if (p) cudaFree(p);
    st->pf_tok = nullptr;
    st->pf_x = st->pf_proj = st->pf_o = st->pf_part = st->pf_ql = st->pf_ol = st->pf_y = st->pf_rlog = st->pf_score = st->pf_logits = nullptr;
    st->pf_mix = st->pf_h = st->pf_io = st->pf_act = st->pf_gx = st->pf_ga = st->pf_qi = st->pf_k = st->pf_v = nullptr;
    st->pf_idx = st->pf_slot = st->pf_count = st->pf_offset = st->pf_bg = st->pf_nb = st->pf_rows = nullptr;
    st->cap = 0;
    st->kv_rows = 0;
}

}  // namespace

int lb_stack_max_lanes(const LbStack* st) {
    int m = lb_dense_gemv_max_tokens(st->d.width, st->d.dtype);
    for (auto& l : st->layers) {
        m = std::min(m, lb_dense_gemv_max_tokens(hv_of(l.s), st->d.dtype));
        if (l.s.ffn == LOOM_B200_FFN_DENSE || l.s.ffn == LOOM_B200_FFN_GATED) m = std::min(m, lb_dense_gemv_max_tokens(l.s.ff, st->d.dtype));
    }
    return m;
}

int lb_stack_ready(loom_b200_ctx* ctx, LbStack* st) {
    LB_REQUIRE(ctx, st->head, "decoder: embeddings and head are not set");
    for (size_t i = 0; i < st->layers.size(); ++i) LB_REQUIRE(ctx, st->layers[i].ready, "decoder: layer %zu has no weights", i);
    return ensure_step_scratch(ctx, st);
}

void lb_stack_free(LbStack* st) {
    if (!st) return;
    free_block(st);
    for (auto& l : st->layers) {
        void* ptrs[] = {l.scal, l.norm1_w, l.norm2_w, l.mixer_norm, l.decay_wt, l.decay_b, l.conv_w, l.bias, l.bias_log2, l.a_log, l.dt_bias, l.gate_b_i, l.gate_b_f,
                        l.conv_ring, l.state, l.mem_norm, l.mem_top, l.k_cache, l.vt_cache, l.latent};
        for (void* p : ptrs)
            if (p) cudaFree(p);
    }
    void* ptrs[] = {st->scal, st->final_w, st->attn_count, st->y, st->x, st->proj, st->o, st->mid, st->ql, st->ol, st->rlog, st->pairs, st->list, st->attn_part};
    for (void* p : ptrs)
        if (p) cudaFree(p);
    delete st;
}

int lb_stack_set_layer(loom_b200_ctx* ctx, LbStack* st, int layer, const loom_b200_layer_spec& s, const loom_b200_layer_weights& w, int lanes) {
    const loom_b200_stack_dims& d = st->d;
    LB_REQUIRE(ctx, layer >= 0 && layer < (int)st->layers.size(), "set_layer: layer %d out of range", layer);
    LbLayer& l = st->layers[layer];
    LB_REQUIRE(ctx, !l.ready, "set_layer: layer %d is already set", layer);
    LB_REQUIRE(ctx, s.mixer >= LOOM_B200_MIXER_GLA && s.mixer <= LOOM_B200_MIXER_MLSTM, "set_layer: mixer %d", s.mixer);
    LB_REQUIRE(ctx, s.heads > 0 && s.dim > 0 && s.vdim > 0, "set_layer: layer %d: heads %d, dim %d, vdim %d", layer, s.heads, s.dim, s.vdim);
    LB_REQUIRE(ctx, s.rank > 0 || s.mixer > LOOM_B200_MIXER_LATENT, "set_layer: layer %d: rank %d", layer, s.rank);
    if (s.mixer == LOOM_B200_MIXER_ATTENTION || s.mixer == LOOM_B200_MIXER_DELTA)
        LB_REQUIRE(ctx, s.kv_heads > 0 && s.heads % s.kv_heads == 0, "set_layer: layer %d: %d heads over %d key heads", layer, s.heads, s.kv_heads);
    auto shaped = [&](const loom_b200_matrix* m, const char* name, int rows, int cols, int groups) -> int {
        LB_REQUIRE(ctx, m != nullptr, "set_layer: layer %d has no matrix '%s'", layer, name);
        LB_REQUIRE(ctx, m->rows == rows && m->cols == cols && m->groups == groups && m->dtype == d.dtype,
                   "set_layer: layer %d: '%s' is %dx%d (%d groups, dtype %d), expected %dx%d (%d groups, dtype %d)", layer, name, m->rows, m->cols, m->groups,
                   m->dtype, rows, cols, groups, d.dtype);
        LB_REQUIRE(ctx, m->device == ctx->device, "set_layer: layer %d: '%s' lives on device %d", layer, name, m->device);
        return 0;
    };
    const int HD = s.heads * s.dim, HV = s.heads * s.vdim;
    int in_rows = 0;
    if (s.mixer == LOOM_B200_MIXER_GLA) {
        LB_REQUIRE(ctx, s.tau > 0, "set_layer: layer %d: tau %g", layer, s.tau);
        LB_REQUIRE(ctx, lb_gla_chunk(s.dim, s.rank) > 0, "set_layer: layer %d: %d key channels with decay rank %d", layer, s.dim, s.rank);
        LB_REQUIRE(ctx, w.mixer_norm && w.decay_w && w.decay_b, "set_layer: layer %d has no head norm or decay weights", layer);
        in_rows = 2 * HD + 2 * HV + s.rank;
    } else if (s.mixer == LOOM_B200_MIXER_ATTENTION) {
        LB_REQUIRE(ctx, s.chunk >= 0, "set_layer: layer %d: chunks of %d positions", layer, s.chunk);
        LB_REQUIRE(ctx, s.buckets == 0 || (w.rel && s.buckets >= 2 && s.bias_max > s.buckets / 2 && s.bias_max < 1e6), "set_layer: layer %d: %d distance buckets up to %g", layer, s.buckets,
                   s.bias_max);
        in_rows = HD + s.kv_heads * (s.dim + s.vdim) + (s.head_gate ? s.heads : 0);
    } else if (s.mixer == LOOM_B200_MIXER_DELTA) {
        LB_REQUIRE(ctx, lb_delta_chunk(s.dim) > 0, "set_layer: layer %d: %d key channels", layer, s.dim);
        LB_REQUIRE(ctx, s.conv >= 1 && s.conv <= 16, "set_layer: layer %d: %d convolution taps (1..16)", layer, s.conv);
        LB_REQUIRE(ctx, w.mixer_norm && w.conv_qkv && w.a_log && w.dt_bias, "set_layer: layer %d has no head norm, convolutions or decay weights", layer);
        LB_REQUIRE(ctx, !w.conv_w, "set_layer: layer %d: the delta rule has convolutions of its own", layer);
        in_rows = 2 * s.kv_heads * s.dim + 2 * HV + 2 * s.heads;
    } else if (s.mixer == LOOM_B200_MIXER_MLSTM) {
        LB_REQUIRE(ctx, lb_memory_chunk(s.dim) > 0, "set_layer: layer %d: %d key channels", layer, s.dim);
        LB_REQUIRE(ctx, s.gate_cap > 0, "set_layer: layer %d: gate cap %g", layer, s.gate_cap);
        LB_REQUIRE(ctx, w.mixer_norm && w.gate_b_i && w.gate_b_f, "set_layer: layer %d has no head norm or gate biases", layer);
        in_rows = 2 * HD + 2 * HV + 2 * s.heads;
    } else {
        const int chunks = lb_slices_of(s.rank, d.dtype) * 8;
        LB_REQUIRE(ctx, chunks <= 256, "set_layer: layer %d: latent size %d", layer, s.rank);
        if (s.kv_from >= 0) {
            LB_REQUIRE(ctx, s.kv_from < layer, "set_layer: layer %d reads the latents of layer %d, which does not come before it", layer, s.kv_from);
            const LbLayer& src = st->layers[s.kv_from];
            LB_REQUIRE(ctx, src.ready && src.latent, "set_layer: layer %d reads the latents of layer %d, which has none of its own", layer, s.kv_from);
            LB_REQUIRE(ctx, src.s.rank == s.rank, "set_layer: layer %d: latent size %d, layer %d has %d", layer, s.rank, s.kv_from, src.s.rank);
        } else {
            LB_REQUIRE(ctx, w.mixer_norm, "set_layer: layer %d has no latent norm", layer);
        }
        in_rows = HD + (s.kv_from >= 0 ? 0 : s.rank);
        if (int rc = shaped(w.up_k, "up_k", HD, s.rank, 1)) return rc;
        if (int rc = shaped(w.up_v, "up_v", HV, s.rank, 1)) return rc;
    }
    if (int rc = shaped(w.in, "in", in_rows, d.width, 1)) return rc;
    if (int rc = shaped(w.out, "out", d.width, HV, 1)) return rc;
    LB_REQUIRE(ctx, !w.conv_w || d.conv_taps >= 1, "set_layer: layer %d has a convolution but the stack has no taps", layer);
    if (s.ffn == LOOM_B200_FFN_DENSE) {
        LB_REQUIRE(ctx, s.ff > 0, "set_layer: layer %d: ff %d", layer, s.ff);
        if (int rc = shaped(w.up, "up", s.ff, d.width, 1)) return rc;
        if (int rc = shaped(w.down, "down", d.width, s.ff, 1)) return rc;
    } else if (s.ffn == LOOM_B200_FFN_GATED) {
        LB_REQUIRE(ctx, s.ff > 0, "set_layer: layer %d: ff %d", layer, s.ff);
        if (int rc = shaped(w.gate, "gate", s.ff, d.width, 1)) return rc;
        if (int rc = shaped(w.up, "up", s.ff, d.width, 1)) return rc;
        if (int rc = shaped(w.down, "down", d.width, s.ff, 1)) return rc;
    } else if (s.ffn == LOOM_B200_FFN_MOE) {
        LB_REQUIRE(ctx, s.ff > 0 && s.experts > 0 && s.experts <= 1024 && s.top > 0 && s.top <= kMaxTop && s.top <= s.experts,
                   "set_layer: layer %d: ff %d, %d experts (at most 1024), top %d (at most %d)", layer, s.ff, s.experts, s.top, kMaxTop);
        if (int rc = shaped(w.router, "router", s.experts, d.width, 1)) return rc;
        if (int rc = shaped(w.gate, "gate", s.ff, d.width, s.experts)) return rc;
        if (int rc = shaped(w.up, "up", s.ff, d.width, s.experts)) return rc;
        if (int rc = shaped(w.down, "down", d.width, s.ff, s.experts)) return rc;
    } else {
        LB_REQUIRE(ctx, s.ffn == LOOM_B200_FFN_NONE, "set_layer: layer %d: feed-forward %d", layer, s.ffn);
    }
    LB_REQUIRE(ctx, !w.conv_w || !w.norm1_w, "set_layer: layer %d: a convolution takes a norm with one gain", layer);
    if (d.post_norm) {
        LB_REQUIRE(ctx, !w.conv_w && s.ffn != LOOM_B200_FFN_MOE, "set_layer: layer %d: norms after the sum are not built for routed experts or a convolution in front of the mixer", layer);
        LB_REQUIRE(ctx, w.norm1_w && (s.ffn == LOOM_B200_FFN_NONE || w.norm2_w), "set_layer: layer %d: norms after the sum have weights per column", layer);
    }
    LB_REQUIRE(ctx, !w.norm2_w || s.ffn != LOOM_B200_FFN_MOE, "set_layer: layer %d: routed experts take a norm with one gain", layer);
    l.s = s;
    if (s.mixer != LOOM_B200_MIXER_LATENT) l.s.kv_from = -1;
    l.w = w;
    l.in_cols = in_rows;
    auto put = [&](float** dst, const float* src, size_t n) -> int {
        LB_CUDA(ctx, cudaMalloc((void**)dst, n * 4));
        LB_CUDA(ctx, cudaMemcpyAsync(*dst, src, n * 4, cudaMemcpyHostToDevice, ctx->stream));
        LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
        return 0;
    };
    auto zero = [&](auto** dst, size_t bytes) -> int {
        LB_CUDA(ctx, cudaMalloc((void**)dst, bytes));
        LB_CUDA(ctx, cudaMemsetAsync(*dst, 0, bytes, ctx->stream));
        return 0;
    };
    const float scal[2] = {w.norm1_w ? 1.f : w.norm1, w.norm2_w ? 1.f : w.norm2};
    if (int rc = put(&l.scal, scal, 2)) return rc;
    if (w.conv_w) {
        std::vector<float> t((size_t)d.conv_taps * st->ldx, 0.f);  // transposed: consecutive channels are consecutive in memory
        for (int c = 0; c < d.width; ++c)
            for (int j = 0; j < d.conv_taps; ++j) t[(size_t)j * st->ldx + c] = w.conv_w[(size_t)c * d.conv_taps + j];
        if (int rc = put(&l.conv_w, t.data(), t.size())) return rc;
        if (int rc = zero(&l.conv_ring, (size_t)lanes * d.conv_taps * st->ldx * 4)) return rc;
    }
    if (w.norm1_w)
        if (int rc = put(&l.norm1_w, w.norm1_w, d.width)) return rc;
    if (w.norm2_w)
        if (int rc = put(&l.norm2_w, w.norm2_w, d.width)) return rc;
    if (s.mixer == LOOM_B200_MIXER_GLA || s.mixer == LOOM_B200_MIXER_DELTA || s.mixer == LOOM_B200_MIXER_MLSTM) {
        std::vector<float> n(HV);
        for (int i = 0; i < HV; ++i) n[i] = w.mixer_norm[s.mixer == LOOM_B200_MIXER_MLSTM ? i : i % s.vdim];
        if (int rc = put(&l.mixer_norm, n.data(), HV)) return rc;
        if (int rc = zero(&l.state, (size_t)lanes * HD * s.vdim * 4)) return rc;
    }
    if (s.mixer == LOOM_B200_MIXER_ATTENTION) {
        // positions that have to stay: a chunk and a block of tokens, or all of them
        l.ring = lb_round_up(d.max_seq_len, 128);
        if (s.chunk > 0) l.ring = std::min(l.ring, lb_round_up(std::min(s.chunk, d.max_seq_len) + kStackBlock, 128));
        l.k_lane = lb_attention_k_bytes(s.kv_heads, s.dim, l.ring, d.dtype);
        l.vt_lane = lb_attention_vt_bytes(s.kv_heads, s.vdim, l.ring, d.dtype);
        if (int rc = zero(&l.k_cache, l.k_lane * lanes)) return rc;
        if (int rc = zero(&l.vt_cache, l.vt_lane * lanes)) return rc;
        if (s.buckets > 0)
            if (int rc = put_bias(ctx, l, w.rel)) return rc;
    } else if (s.mixer == LOOM_B200_MIXER_DELTA) {
        const int ch = 2 * s.kv_heads * s.dim + HV;
        std::vector<float> t((size_t)ch * s.conv);  // transposed: consecutive channels are consecutive in memory
        for (int c = 0; c < ch; ++c)
            for (int j = 0; j < s.conv; ++j) t[(size_t)j * ch + c] = w.conv_qkv[(size_t)c * s.conv + j];
        if (int rc = put(&l.conv_w, t.data(), t.size())) return rc;
        if (int rc = zero(&l.conv_ring, (size_t)lanes * s.conv * ch * 4)) return rc;
        if (int rc = put(&l.a_log, w.a_log, s.heads)) return rc;
        if (int rc = put(&l.dt_bias, w.dt_bias, s.heads)) return rc;
    } else if (s.mixer == LOOM_B200_MIXER_MLSTM) {
        if (int rc = put(&l.gate_b_i, w.gate_b_i, s.heads)) return rc;
        if (int rc = put(&l.gate_b_f, w.gate_b_f, s.heads)) return rc;
        if (int rc = zero(&l.mem_norm, (size_t)lanes * 2 * HD * 4)) return rc;
        if (int rc = zero(&l.mem_top, (size_t)lanes * 2 * s.heads * 4)) return rc;
    } else if (s.mixer == LOOM_B200_MIXER_GLA) {
        std::vector<float> t((size_t)HD * s.rank);  // transposed: consecutive channels are consecutive in memory
        for (int c = 0; c < HD; ++c)
            for (int r = 0; r < s.rank; ++r) t[(size_t)r * HD + c] = w.decay_w[(size_t)c * s.rank + r];
        if (int rc = put(&l.decay_wt, t.data(), t.size())) return rc;
        if (int rc = put(&l.decay_b, w.decay_b, HD)) return rc;
    } else if (s.kv_from < 0) {
        if (int rc = put(&l.mixer_norm, w.mixer_norm, s.rank)) return rc;
        l.latent_lane = lb_img_bytes(d.max_seq_len, s.rank, d.dtype);
        if (int rc = zero(&l.latent, l.latent_lane * lanes)) return rc;
    }
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    l.w.mixer_norm = l.w.decay_w = l.w.decay_b = l.w.conv_w = nullptr;  // host pointers of the call
    l.w.norm1_w = l.w.norm2_w = l.w.rel = l.w.conv_qkv = l.w.a_log = l.w.dt_bias = l.w.gate_b_i = l.w.gate_b_f = nullptr;
    l.ready = true;
    st->lanes = lanes;
    return 0;
}

int lb_stack_step(loom_b200_ctx* ctx, LbStack* st, const int* tok, const int* pos, int lane0, int M) {
    const loom_b200_stack_dims& d = st->d;
    const int dt = d.dtype, W = d.width;
    const float eps = (float)d.norm_eps, mult = (float)d.residual_mult;
    LB_REQUIRE(ctx, M >= 1 && M <= lb_stack_max_lanes(st), "stack_step: %d sequences", M);
    if (int rc = embed(ctx, st, tok, M, st->x)) return rc;
    const float* waiting = nullptr;  // norms after the sum: the weights of the norm that st->y waits for
    // the input of a product: the normed residual; with norms after the sum the sum's norm, whose result is the residual
    auto input = [&](LbDenseGemv& g, const float* gain, const float* gain_w) -> int {
        g.K = W;
        g.M = M;
        g.ldx = st->ldx;
        g.eps = eps;
        g.x = st->x;
        if (!d.post_norm) {
            g.gain = gain;
            g.gain_w = gain_w;
            return LB_DPRO_NORM;
        }
        if (!waiting) return LB_DPRO_PLAIN;
        g.x = st->y;
        g.gain_w = waiting;
        g.x_out = st->x;
        return LB_DPRO_NORM;
    };
    auto residual = [&](LbDenseGemv& g) {
        g.out = d.post_norm ? st->y : st->x;
        g.ldo = st->ldx;
        g.res = st->x;
        g.mult = mult;
        g.res_mult = d.post_norm ? (float)d.residual_alpha : 1.f;
    };
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        LbDenseGemv in;
        const int pro = input(in, l.scal, l.norm1_w);
        in.w = l.w.in->data;
        in.rows = l.in_cols;
        in.slices = l.w.in->slices;
        const bool conv = l.conv_w && s.mixer != LOOM_B200_MIXER_DELTA;
        if (conv) {
            in.conv_w = l.conv_w;
            in.conv_ring = l.conv_ring;
            in.taps = d.conv_taps;
            in.ring_ld = st->ldx;
            in.pos = pos;
            in.lane0 = lane0;
        }
        in.out = st->proj;
        in.ldo = st->ldp;
        if (int rc = lb_dense_gemv(ctx, dt, conv ? LB_DPRO_CONV : pro, LB_DEPI_F32, in)) return rc;

        LbDenseGemv out;
        out.w = l.w.out->data;
        out.rows = W;
        out.K = hv_of(s);
        out.slices = l.w.out->slices;
        out.M = M;
        residual(out);
        out.x = st->o;
        out.ldx = st->ldo;
        if (recurrent(s)) {
            int rc = 0;
            if (s.mixer == LOOM_B200_MIXER_GLA)
                rc = lb_gla_step(ctx, gla_of(l, st->proj, st->ldp, st->o, st->ldo, 0), pos, lane0, M);
            else if (s.mixer == LOOM_B200_MIXER_DELTA)
                rc = lb_delta_step(ctx, delta_of(l, st->proj, st->ldp, st->o, st->ldo, 0), pos, lane0, M);
            else
                rc = lb_memory_step(ctx, memory_of(l, st->proj, st->ldp, st->o, st->ldo, 0), pos, lane0, M);
            if (rc) return rc;
            out.gate = st->proj + gate_col(s);
            out.gate_ld = st->ldp;
            out.gate_sigmoid = s.mixer == LOOM_B200_MIXER_MLSTM;
            out.head_w = l.mixer_norm;
            out.head_dim = s.vdim;
            out.eps = eps;
            if ((rc = lb_dense_gemv(ctx, dt, LB_DPRO_GATED, LB_DEPI_RESID, out))) return rc;
        } else if (s.mixer == LOOM_B200_MIXER_ATTENTION) {
            LbAttention a = attention_of(st, l, st->proj, st->ldp);
            a.pos = pos;
            a.lane0 = lane0;
            if (int rc = lb_attention_step(ctx, dt, a, M, st->attn_part, st->attn_count, st->o, st->ldo)) return rc;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_PLAIN, LB_DEPI_RESID, out)) return rc;
        } else {
            LbLatent a = latent_of(st, l, st->proj, st->ldp);
            a.pos = pos;
            a.lane0 = lane0;
            if (int rc = latent_few(ctx, st, dt, a, s.kv_from < 0 ? st->proj + s.heads * s.dim : nullptr, l.mixer_norm, M, st->ql, st->ol, st->attn_part, st->o, st->ldo)) return rc;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_PLAIN, LB_DEPI_RESID, out)) return rc;
        }
        if (d.post_norm) waiting = l.norm1_w;

        if (s.ffn == LOOM_B200_FFN_NONE) continue;
        LbDenseGemv f;
        input(f, l.scal + 1, l.norm2_w);
        LbDenseGemv y;
        y.w = l.w.down->data;
        y.rows = W;
        y.K = s.ff;
        y.slices = l.w.down->slices;
        y.M = M;
        residual(y);
        if (s.ffn == LOOM_B200_FFN_DENSE || s.ffn == LOOM_B200_FFN_GATED) {
            const bool gated = s.ffn == LOOM_B200_FFN_GATED;
            f.w = gated ? l.w.gate->data : l.w.up->data;
            f.w2 = gated ? l.w.up->data : nullptr;
            f.rows = s.ff;
            f.slices = l.w.up->slices;
            f.out = st->mid;
            f.ldo = st->ldm;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_NORM, gated ? LB_DEPI_SILU : LB_DEPI_GELU, f)) return rc;
            y.x = st->mid;
            y.ldx = st->ldm;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_PLAIN, LB_DEPI_RESID, y)) return rc;
        } else {
            f.w = l.w.router->data;
            f.rows = s.experts;
            f.slices = l.w.router->slices;
            f.out = st->rlog;
            f.ldo = st->ldr;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_NORM, LB_DEPI_F32, f)) return rc;
            const int lde = l.w.down->slices * lb_slice_cols(dt);
            f.w = l.w.gate->data;
            f.w2 = l.w.up->data;
            f.group_bytes = l.w.gate->group_bytes;
            f.rows = s.ff;
            f.slices = l.w.gate->slices;
            f.logits = st->rlog;
            f.ldl = st->ldr;
            f.experts = s.experts;
            f.top = s.top;
            f.list = st->list;
            f.out = nullptr;
            f.out_pairs = st->pairs;
            f.ldo = lde;
            f.limit = (float)s.limit;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_MOE, LB_DEPI_GLU, f)) return rc;
            y.group_bytes = l.w.down->group_bytes;
            y.list = st->list;
            y.pairs = st->pairs;
            y.ldp = lde;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_PAIRS, LB_DEPI_RESID, y)) return rc;
        }
        if (d.post_norm) waiting = l.norm2_w;
    }
    if (!d.post_norm) return 0;
    LbNormBlock n;
    n.x = st->y;
    n.ldx = st->ldx;
    n.T = M;
    n.width = W;
    n.slices = lb_slices_of(W, dt);
    n.gain_w = waiting;
    n.rows = st->x;
    n.eps = eps;
    return lb_norm_block(ctx, dt, n);
}

int lb_stack_ensure_block(loom_b200_ctx* ctx, LbStack* st, int tokens) {
    if (tokens <= st->cap) return 0;
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "stack scratch would grow while recording a graph");
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    free_block(st);
    const int dt = st->d.dtype, T = lb_round_up(tokens, kImgRows), W = st->d.width;
    size_t o = 0, io = 0, mix = 0, hr = 0, qi = 0, act = 0, gx = 0, ga = 0, y = 0, rl = 0, pairs = 0, ex = 0, nb = 0;
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        o = std::max(o, (size_t)T * lb_round_up(hv_of(s), 8));
        io = std::max(io, lb_img_bytes(T, hv_of(s), dt));
        MixerScratch m;
        mix = std::max(mix, mixer_scratch(l, T, nullptr, m));
        if (s.mixer == LOOM_B200_MIXER_LATENT) {
            hr = std::max(hr, (size_t)std::min(T, kLatentStepTokens) * s.heads * s.rank);
            qi = std::max(qi, lb_latent_heads_bytes(latent_of(st, l, nullptr, 0), T));
        }
        if (s.mixer == LOOM_B200_MIXER_ATTENTION) qi = std::max(qi, lb_attention_q_bytes(attention_of(st, l, nullptr, 0), T));
        if (s.ffn == LOOM_B200_FFN_DENSE || s.ffn == LOOM_B200_FFN_GATED) act = std::max(act, lb_img_bytes(T, s.ff, dt));
        if (s.ffn == LOOM_B200_FFN_MOE) {
            const int b = lb_route_max_blocks(T, s.experts, s.top);
            gx = std::max(gx, lb_img_bytes(b * kImgRows, W, dt));
            ga = std::max(ga, lb_img_bytes(b * kImgRows, s.ff, dt));
            y = std::max(y, (size_t)b * kImgRows * st->ldx);
            rl = std::max(rl, (size_t)T * lb_round_up(s.experts, 8));
            pairs = std::max(pairs, (size_t)T * s.top);
            ex = std::max(ex, (size_t)s.experts);
            nb = std::max(nb, (size_t)b);
        }
    }
    st->ldl = lb_round_up(st->d.vocab, 8);
    auto A = [&](auto** p, size_t bytes) -> int {
        if (bytes == 0) return 0;
        LB_CUDA(ctx, cudaMalloc((void**)p, bytes));
        LB_CUDA(ctx, cudaMemsetAsync(*p, 0, bytes, ctx->stream));
        return 0;
    };
#define LB_A(p, bytes) \
    if (int rc = A(&st->p, (bytes))) return rc
    LB_A(pf_tok, (size_t)T * 4);
    LB_A(pf_x, (size_t)T * st->ldx * 4);
    LB_A(pf_h, lb_img_bytes(T, W, dt));
    LB_A(pf_proj, (size_t)T * st->ldp * 4);
    LB_A(pf_o, o * 4);
    LB_A(pf_io, io);
    LB_A(pf_mix, mix);
    LB_A(pf_part, attn_part_elems(ctx, st, T) * 4);
    if (is_bf16(st)) LB_A(pf_qi, qi);
    LB_A(pf_ql, hr * 4);
    LB_A(pf_ol, hr * 4);
    LB_A(pf_act, act);
    LB_A(pf_gx, gx);
    LB_A(pf_ga, ga);
    LB_A(pf_y, y * 4);
    LB_A(pf_rlog, rl * 4);
    LB_A(pf_idx, pairs * 4);
    LB_A(pf_slot, pairs * 4);
    LB_A(pf_score, pairs * 4);
    LB_A(pf_count, ex * 4);
    LB_A(pf_offset, ex * 4);
    LB_A(pf_bg, nb * 4);
    LB_A(pf_nb, 4);
    LB_A(pf_rows, (size_t)T * 4);
    LB_A(pf_logits, (size_t)kStackHeadRows * st->ldl * 4);
#undef LB_A
    st->cap = T;
    return 0;
}

int lb_stack_block(loom_b200_ctx* ctx, LbStack* st, int T, int pos0, int lane) {
    const loom_b200_stack_dims& d = st->d;
    const int dt = d.dtype, W = d.width, slices = lb_slices_of(W, dt);
    const float eps = (float)d.norm_eps, mult = (float)d.residual_mult;
    LB_REQUIRE(ctx, T >= 1 && T <= st->cap, "stack_block: %d tokens", T);
    if (int rc = embed(ctx, st, st->pf_tok, T, st->pf_x)) return rc;
    const float res_mult = d.post_norm ? (float)d.residual_alpha : 1.f;
    if (d.post_norm)
        if (int rc = lb_rows_image(ctx, dt, st->pf_x, st->ldx, T, W, slices, st->pf_h)) return rc;
    // norms after the sum: in place, with the next product's input
    auto normed = [&](const float* gain_w) {
        LbNormBlock n;
        n.x = n.rows = st->pf_x;
        n.ldx = st->ldx;
        n.T = T;
        n.width = W;
        n.slices = slices;
        n.gain_w = gain_w;
        n.eps = eps;
        n.img = st->pf_h;
        return lb_norm_block(ctx, dt, n);
    };
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        LbNormBlock n;
        n.x = st->pf_x;
        n.ldx = st->ldx;
        n.T = T;
        n.width = W;
        n.slices = slices;
        n.gain = l.scal;
        n.gain_w = l.norm1_w;
        n.eps = eps;
        n.img = st->pf_h;
        const bool conv = l.conv_w && s.mixer != LOOM_B200_MIXER_DELTA;
        if (conv) {
            n.conv_w = l.conv_w;
            n.taps = d.conv_taps;
            n.ring_ld = st->ldx;
            n.ring = l.conv_ring + (size_t)lane * d.conv_taps * st->ldx;
            n.pos0 = pos0;
        }
        if (!d.post_norm)
            if (int rc = lb_norm_block(ctx, dt, n)) return rc;
        if (conv)
            if (int rc = lb_conv_commit(ctx, n)) return rc;
        LbDenseGemm g;
        g.x = st->pf_h;
        g.tokens = T;
        g.w = l.w.in->data;
        g.rows = l.in_cols;
        g.slices = slices;
        g.out = st->pf_proj;
        g.ldo = st->ldp;
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_F32, g)) return rc;

        const int hv = hv_of(s), ldo = lb_round_up(hv, 8), oslices = l.w.out->slices;
        if (recurrent(s)) {
            MixerScratch m;
            mixer_scratch(l, T, st->pf_mix, m);
            int rc = 0;
            if (s.mixer == LOOM_B200_MIXER_GLA)
                rc = lb_gla_block(ctx, gla_of(l, st->pf_proj, st->ldp, st->pf_o, ldo, lane), m.c, T, pos0);
            else if (s.mixer == LOOM_B200_MIXER_DELTA)
                rc = lb_delta_block(ctx, delta_of(l, st->pf_proj, st->ldp, st->pf_o, ldo, lane), m.delta, T, pos0);
            else
                rc = lb_memory_block(ctx, memory_of(l, st->pf_proj, st->ldp, st->pf_o, ldo, lane), m.mem, T, pos0);
            if (rc) return rc;
            const bool mem = s.mixer == LOOM_B200_MIXER_MLSTM;
            if ((rc = lb_gated_heads_image(ctx, dt, st->pf_o, ldo, st->pf_proj + gate_col(s), st->ldp, T, s.heads, s.vdim, l.mixer_norm, mem, mem ? m.mem.scale : nullptr, eps,
                                           oslices, st->pf_io)))
                return rc;
        } else if (s.mixer == LOOM_B200_MIXER_ATTENTION) {
            LbAttention a = attention_of(st, l, st->pf_proj, st->ldp);
            a.pos0 = pos0;
            a.lane0 = lane;
            const bool tc = attention_step_tokens(st, l, T) < T;
            if (int rc = lb_attention_store(ctx, dt, a, T, tc ? st->pf_qi : nullptr)) return rc;
            if (tc) {
                if (int rc = lb_attention_block(ctx, a, T, st->pf_qi, st->pf_io, oslices)) return rc;
            } else {
                if (int rc = lb_attention_step(ctx, dt, a, T, st->pf_part, st->attn_count, st->pf_o, ldo)) return rc;
                if (int rc = lb_rows_image(ctx, dt, st->pf_o, ldo, T, hv, oslices, st->pf_io)) return rc;
            }
        } else {
            LbLatent a = latent_of(st, l, st->pf_proj, st->ldp);
            a.pos0 = pos0;
            a.lane0 = lane;
            if (s.kv_from < 0)
                if (int rc = lb_latent_store(ctx, dt, a, st->pf_proj + s.heads * s.dim, st->ldp, l.mixer_norm, eps, T)) return rc;
            if (dt == LOOM_B200_DTYPE_BF16 && T > kLatentStepTokens && lb_latent_block_supported(a)) {
                if (int rc = ensure_kv(ctx, st, pos0 + T)) return rc;
                if (int rc = lb_latent_block(ctx, a, T, st->pf_qi, st->pf_k, st->pf_v, lb_ceil_div((int)st->kv_rows, 64), st->pf_io, oslices)) return rc;
            } else {
                // a few tokens at a time through the step's kernels, so that the scratch stays small
                for (int t0 = 0; t0 < T; t0 += kLatentStepTokens) {
                    LbLatent c = a;
                    const int n = std::min(kLatentStepTokens, T - t0);
                    c.q = a.q + (size_t)t0 * a.ldq;
                    c.pos0 = pos0 + t0;
                    if (int rc = latent_few(ctx, st, dt, c, nullptr, nullptr, n, st->pf_ql, st->pf_ol, st->pf_part, st->pf_o + (size_t)t0 * ldo, ldo)) return rc;
                }
                if (int rc = lb_rows_image(ctx, dt, st->pf_o, ldo, T, hv, oslices, st->pf_io)) return rc;
            }
        }
        g = LbDenseGemm();
        g.x = st->pf_io;
        g.tokens = T;
        g.w = l.w.out->data;
        g.rows = W;
        g.slices = oslices;
        g.out = st->pf_x;
        g.ldo = st->ldx;
        g.mult = mult;
        g.res_mult = res_mult;
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_RESID, g)) return rc;
        if (d.post_norm)
            if (int rc = normed(l.norm1_w)) return rc;

        if (s.ffn == LOOM_B200_FFN_NONE) continue;
        n.conv_w = nullptr;
        n.taps = 1;
        n.gain = l.scal + 1;
        n.gain_w = l.norm2_w;
        if (!d.post_norm)
            if (int rc = lb_norm_block(ctx, dt, n)) return rc;
        g = LbDenseGemm();
        g.x = st->pf_h;
        g.tokens = T;
        g.slices = slices;
        if (s.ffn == LOOM_B200_FFN_DENSE || s.ffn == LOOM_B200_FFN_GATED) {
            const bool gated = s.ffn == LOOM_B200_FFN_GATED;
            g.w = gated ? l.w.gate->data : l.w.up->data;
            g.w2 = gated ? l.w.up->data : nullptr;
            g.rows = s.ff;
            g.img = st->pf_act;
            g.img_slices = l.w.down->slices;
            if (int rc = lb_dense_gemm(ctx, dt, gated ? LB_DEPI_SILU : LB_DEPI_GELU, g)) return rc;
            g = LbDenseGemm();
            g.x = st->pf_act;
            g.tokens = T;
            g.w = l.w.down->data;
            g.rows = W;
            g.slices = l.w.down->slices;
            g.out = st->pf_x;
            g.ldo = st->ldx;
            g.mult = mult;
            g.res_mult = res_mult;
            if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_RESID, g)) return rc;
            if (d.post_norm)
                if (int rc = normed(l.norm2_w)) return rc;
            continue;
        }
        g.w = l.w.router->data;
        g.rows = s.experts;
        g.out = st->pf_rlog;
        g.ldo = lb_round_up(s.experts, 8);
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_F32, g)) return rc;
        LbRouteBlock r;
        r.T = T;
        r.experts = s.experts;
        r.top = s.top;
        r.logits = st->pf_rlog;
        r.ldl = g.ldo;
        r.idx = st->pf_idx;
        r.score = st->pf_score;
        r.slot = st->pf_slot;
        r.count = st->pf_count;
        r.offset = st->pf_offset;
        r.block_group = st->pf_bg;
        r.nblocks = st->pf_nb;
        if (int rc = lb_route_block(ctx, r)) return rc;
        if (int rc = lb_route_gather(ctx, dt, r, st->pf_x, st->ldx, W, l.scal + 1, eps, slices, st->pf_gx)) return rc;
        g = LbDenseGemm();
        g.nblocks = st->pf_nb;
        g.block_group = st->pf_bg;
        g.max_blocks = lb_route_max_blocks(T, s.experts, s.top);
        g.x = st->pf_gx;
        g.w = l.w.gate->data;
        g.w2 = l.w.up->data;
        g.group_bytes = l.w.gate->group_bytes;
        g.rows = s.ff;
        g.slices = slices;
        g.img = st->pf_ga;
        g.img_slices = l.w.down->slices;
        g.limit = (float)s.limit;
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_GLU, g)) return rc;
        g.x = st->pf_ga;
        g.w = l.w.down->data;
        g.w2 = nullptr;
        g.group_bytes = l.w.down->group_bytes;
        g.rows = W;
        g.slices = l.w.down->slices;
        g.out = st->pf_y;
        g.ldo = st->ldx;
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_F32, g)) return rc;
        if (int rc = lb_route_combine(ctx, r, st->pf_y, st->ldx, mult, W, st->pf_x, st->ldx)) return rc;
    }
    return 0;
}

int lb_stack_head(loom_b200_ctx* ctx, LbStack* st, const float* x, const int* rows_dev, int n, float* out, int ldo) {
    LbDenseGemv h;
    h.w = st->head->data;
    h.rows = st->d.vocab;
    h.K = st->d.width;
    h.slices = st->head->slices;
    h.M = n;
    h.x = x;
    h.ldx = st->ldx;
    h.row_idx = rows_dev;
    h.gain = st->final_w ? nullptr : st->scal + 1;
    h.gain_w = st->final_w;
    h.eps = (float)st->d.norm_eps;
    h.out = out;
    h.ldo = ldo;
    return lb_dense_gemv(ctx, st->d.dtype, LB_DPRO_NORM, LB_DEPI_F32, h);
}

int lb_stack_head_block(loom_b200_ctx* ctx, LbStack* st, int n) {
    LB_REQUIRE(ctx, n >= 1 && n <= kStackHeadRows, "stack_head_block: %d rows", n);
    LbNormBlock b;
    b.x = st->pf_x;
    b.ldx = st->ldx;
    b.row_idx = st->pf_rows;
    b.T = n;
    b.width = st->d.width;
    b.slices = st->head->slices;
    b.gain = st->final_w ? nullptr : st->scal + 1;
    b.gain_w = st->final_w;
    b.eps = (float)st->d.norm_eps;
    b.img = st->pf_h;
    if (int rc = lb_norm_block(ctx, st->d.dtype, b)) return rc;
    LbDenseGemm g;
    g.x = st->pf_h;
    g.tokens = n;
    g.w = st->head->data;
    g.rows = st->d.vocab;
    g.slices = st->head->slices;
    g.out = st->pf_logits;
    g.ldo = st->ldl;
    return lb_dense_gemm(ctx, st->d.dtype, LB_DEPI_F32, g);
}
