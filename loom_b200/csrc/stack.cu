// stack.cu -- the layers of a stack decoder: weights and states per layer, the one-token-per-sequence step and the token block.
//
// Step, per layer (M <= 8 sequences, one token each; every launch chained by programmatic dependent launch):
//   gated linear attention   {norm + short convolution + input projections} -> {decay, state update, read-out}
//                            -> {per-head norm, gate, output projection, residual}
//   latent attention         {norm + short convolution + query / latent projections} -> {queries into latent space, latent
//                            norm, cache} -> {attention over the latents} -> {values} -> {output projection, residual}
//   feed-forward             dense {norm, up, gelu} -> {down, residual}; routed {norm, router} -> {choice, norm, gate / up,
//                            clamped unit} -> {down of every chosen expert, sum, residual}
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
    g.state = l.gla_state + (size_t)lane * s.heads * s.dim * s.vdim;
    g.o = o;
    g.ldo = ldo;
    return g;
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

// floats of the split results of up to `tokens` tokens of any latent layer
size_t latent_part_elems(loom_b200_ctx* ctx, LbStack* st, int tokens) {
    size_t n = 0;
    for (auto& l : st->layers) {
        if (l.s.mixer != LOOM_B200_MIXER_LATENT || !is_bf16(st)) continue;
        const LbLatent a = latent_of(st, l, nullptr, 0);
        for (int t = 1; t <= tokens; ++t) n = std::max(n, (size_t)t * l.s.heads * lb_latent_step_splits(ctx, a, t) * (l.s.rank + 2));
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
    for (auto& l : st->layers) {
        in_cols = std::max(in_cols, l.in_cols);
        hv = std::max(hv, hv_of(l.s));
        if (l.s.mixer == LOOM_B200_MIXER_LATENT) hr = std::max(hr, l.s.heads * l.s.rank);
        if (l.s.ffn == LOOM_B200_FFN_DENSE) ff = std::max(ff, l.s.ff);
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
    if (int rc = A(&st->proj, (size_t)M * st->ldp * 4)) return rc;
    if (int rc = A(&st->o, (size_t)M * st->ldo * 4)) return rc;
    if (int rc = A(&st->mid, (size_t)M * st->ldm * 4)) return rc;
    if (int rc = A(&st->ql, (size_t)M * hr * 4)) return rc;
    if (int rc = A(&st->ol, (size_t)M * hr * 4)) return rc;
    if (int rc = A(&st->rlog, (size_t)M * st->ldr * 4)) return rc;
    if (int rc = A(&st->attn_part, latent_part_elems(ctx, st, M) * 4)) return rc;
    if (int rc = A(&st->pairs, (size_t)M * top * eff * (is_bf16(st) ? 2 : 4))) return rc;
    if (int rc = A(&st->list, sizeof(LbRouteList))) return rc;
    st->scratch_ready = true;
    return 0;
}

void free_block(LbStack* st) {
    void* ptrs[] = {st->pf_tok, st->pf_x, st->pf_proj, st->pf_o, st->pf_qd, st->pf_kd, st->pf_cw, st->pf_part, st->pf_cs, st->pf_cd, st->pf_ql, st->pf_ol, st->pf_y, st->pf_rlog,
                    st->pf_score, st->pf_logits, st->pf_h, st->pf_io, st->pf_act, st->pf_gx, st->pf_ga, st->pf_idx, st->pf_slot, st->pf_count,
                    st->pf_offset, st->pf_bg, st->pf_nb, st->pf_rows, st->pf_qi, st->pf_k, st->pf_v};
    for (void* p : ptrs)
        if (p) cudaFree(p);
    st->pf_tok = nullptr;
    st->pf_x = st->pf_proj = st->pf_o = st->pf_qd = st->pf_kd = st->pf_cw = st->pf_part = st->pf_cs = st->pf_cd = st->pf_ql = st->pf_ol = st->pf_y = st->pf_rlog = st->pf_score = st->pf_logits = nullptr;
    st->pf_h = st->pf_io = st->pf_act = st->pf_gx = st->pf_ga = st->pf_qi = st->pf_k = st->pf_v = nullptr;
    st->pf_idx = st->pf_slot = st->pf_count = st->pf_offset = st->pf_bg = st->pf_nb = st->pf_rows = nullptr;
    st->cap = 0;
    st->kv_rows = 0;
}

}  // namespace

int lb_stack_max_lanes(const LbStack* st) {
    int m = lb_dense_gemv_max_tokens(st->d.width, st->d.dtype);
    for (auto& l : st->layers) {
        m = std::min(m, lb_dense_gemv_max_tokens(hv_of(l.s), st->d.dtype));
        if (l.s.ffn == LOOM_B200_FFN_DENSE) m = std::min(m, lb_dense_gemv_max_tokens(l.s.ff, st->d.dtype));
    }
    return m;
}

int lb_stack_ready(loom_b200_ctx* ctx, LbStack* st) {
    LB_REQUIRE(ctx, st->table && st->head, "decoder: embeddings and head are not set");
    for (size_t i = 0; i < st->layers.size(); ++i) LB_REQUIRE(ctx, st->layers[i].ready, "decoder: layer %zu has no weights", i);
    return ensure_step_scratch(ctx, st);
}

void lb_stack_free(LbStack* st) {
    if (!st) return;
    free_block(st);
    for (auto& l : st->layers) {
        void* ptrs[] = {l.scal, l.mixer_norm, l.decay_wt, l.decay_b, l.conv_w, l.conv_ring, l.gla_state, l.latent};
        for (void* p : ptrs)
            if (p) cudaFree(p);
    }
    void* ptrs[] = {st->scal, st->x, st->proj, st->o, st->mid, st->ql, st->ol, st->rlog, st->pairs, st->list, st->attn_part};
    for (void* p : ptrs)
        if (p) cudaFree(p);
    delete st;
}

int lb_stack_set_layer(loom_b200_ctx* ctx, LbStack* st, int layer, const loom_b200_layer_spec& s, const loom_b200_layer_weights& w, int lanes) {
    const loom_b200_stack_dims& d = st->d;
    LB_REQUIRE(ctx, layer >= 0 && layer < (int)st->layers.size(), "set_layer: layer %d out of range", layer);
    LbLayer& l = st->layers[layer];
    LB_REQUIRE(ctx, !l.ready, "set_layer: layer %d is already set", layer);
    LB_REQUIRE(ctx, s.mixer == LOOM_B200_MIXER_GLA || s.mixer == LOOM_B200_MIXER_LATENT, "set_layer: mixer %d", s.mixer);
    LB_REQUIRE(ctx, s.heads > 0 && s.dim > 0 && s.vdim > 0 && s.rank > 0, "set_layer: layer %d: heads %d, dim %d, vdim %d, rank %d", layer, s.heads, s.dim, s.vdim, s.rank);
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
    const float scal[2] = {w.norm1, w.norm2};
    if (int rc = put(&l.scal, scal, 2)) return rc;
    if (w.conv_w) {
        std::vector<float> t((size_t)d.conv_taps * st->ldx, 0.f);  // transposed: consecutive channels are consecutive in memory
        for (int c = 0; c < d.width; ++c)
            for (int j = 0; j < d.conv_taps; ++j) t[(size_t)j * st->ldx + c] = w.conv_w[(size_t)c * d.conv_taps + j];
        if (int rc = put(&l.conv_w, t.data(), t.size())) return rc;
        if (int rc = zero(&l.conv_ring, (size_t)lanes * d.conv_taps * st->ldx * 4)) return rc;
    }
    if (s.mixer == LOOM_B200_MIXER_GLA) {
        if (int rc = put(&l.mixer_norm, w.mixer_norm, s.vdim)) return rc;
        std::vector<float> t((size_t)HD * s.rank);  // transposed: consecutive channels are consecutive in memory
        for (int c = 0; c < HD; ++c)
            for (int r = 0; r < s.rank; ++r) t[(size_t)r * HD + c] = w.decay_w[(size_t)c * s.rank + r];
        if (int rc = put(&l.decay_wt, t.data(), t.size())) return rc;
        if (int rc = put(&l.decay_b, w.decay_b, HD)) return rc;
        if (int rc = zero(&l.gla_state, (size_t)lanes * HD * s.vdim * 4)) return rc;
    } else if (s.kv_from < 0) {
        if (int rc = put(&l.mixer_norm, w.mixer_norm, s.rank)) return rc;
        l.latent_lane = lb_img_bytes(d.max_seq_len, s.rank, d.dtype);
        if (int rc = zero(&l.latent, l.latent_lane * lanes)) return rc;
    }
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    l.w.mixer_norm = l.w.decay_w = l.w.decay_b = l.w.conv_w = nullptr;  // host pointers of the call
    l.ready = true;
    st->lanes = lanes;
    return 0;
}

int lb_stack_step(loom_b200_ctx* ctx, LbStack* st, const int* tok, const int* pos, int lane0, int M) {
    const loom_b200_stack_dims& d = st->d;
    const int dt = d.dtype, W = d.width;
    const float eps = (float)d.norm_eps, mult = (float)d.residual_mult;
    LB_REQUIRE(ctx, M >= 1 && M <= lb_stack_max_lanes(st), "stack_step: %d sequences", M);
    if (int rc = lb_embed_norm(ctx, dt, st->table, d.vocab, W, tok, M, st->scal, eps, st->x, st->ldx)) return rc;
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        LbDenseGemv in;
        in.w = l.w.in->data;
        in.rows = l.in_cols;
        in.K = W;
        in.slices = l.w.in->slices;
        in.M = M;
        in.x = st->x;
        in.ldx = st->ldx;
        in.gain = l.scal;
        in.eps = eps;
        in.conv_w = l.conv_w;
        in.conv_ring = l.conv_ring;
        in.taps = d.conv_taps;
        in.ring_ld = st->ldx;
        in.pos = pos;
        in.lane0 = lane0;
        in.out = st->proj;
        in.ldo = st->ldp;
        if (int rc = lb_dense_gemv(ctx, dt, l.conv_w ? LB_DPRO_CONV : LB_DPRO_NORM, LB_DEPI_F32, in)) return rc;

        LbDenseGemv out;
        out.w = l.w.out->data;
        out.rows = W;
        out.K = hv_of(s);
        out.slices = l.w.out->slices;
        out.M = M;
        out.out = st->x;
        out.ldo = st->ldx;
        out.mult = mult;
        if (s.mixer == LOOM_B200_MIXER_GLA) {
            LbGla g = gla_of(l, st->proj, st->ldp, st->o, st->ldo, 0);
            if (int rc = lb_gla_step(ctx, g, pos, lane0, M)) return rc;
            out.x = st->o;
            out.ldx = st->ldo;
            out.gate = st->proj + 2 * s.heads * s.dim + hv_of(s);
            out.gate_ld = st->ldp;
            out.head_w = l.mixer_norm;
            out.head_dim = s.vdim;
            out.eps = eps;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_GATED, LB_DEPI_RESID, out)) return rc;
        } else {
            LbLatent a = latent_of(st, l, st->proj, st->ldp);
            a.pos = pos;
            a.lane0 = lane0;
            if (int rc = latent_few(ctx, st, dt, a, s.kv_from < 0 ? st->proj + s.heads * s.dim : nullptr, l.mixer_norm, M, st->ql, st->ol, st->attn_part, st->o, st->ldo)) return rc;
            out.x = st->o;
            out.ldx = st->ldo;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_PLAIN, LB_DEPI_RESID, out)) return rc;
        }

        if (s.ffn == LOOM_B200_FFN_NONE) continue;
        LbDenseGemv f;
        f.K = W;
        f.M = M;
        f.x = st->x;
        f.ldx = st->ldx;
        f.gain = l.scal + 1;
        f.eps = eps;
        LbDenseGemv y;
        y.w = l.w.down->data;
        y.rows = W;
        y.K = s.ff;
        y.slices = l.w.down->slices;
        y.M = M;
        y.out = st->x;
        y.ldo = st->ldx;
        y.mult = mult;
        if (s.ffn == LOOM_B200_FFN_DENSE) {
            f.w = l.w.up->data;
            f.rows = s.ff;
            f.slices = l.w.up->slices;
            f.out = st->mid;
            f.ldo = st->ldm;
            if (int rc = lb_dense_gemv(ctx, dt, LB_DPRO_NORM, LB_DEPI_GELU, f)) return rc;
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
    }
    return 0;
}

int lb_stack_ensure_block(loom_b200_ctx* ctx, LbStack* st, int tokens) {
    if (tokens <= st->cap) return 0;
    if (ctx->capturing) return lb_fail(ctx, LOOM_B200_ERR_INVALID, "stack scratch would grow while recording a graph");
    LB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
    free_block(st);
    const int dt = st->d.dtype, T = lb_round_up(tokens, kImgRows), W = st->d.width;
    size_t o = 0, io = 0, qd = 0, cs = 0, cd = 0, cw = 0, hr = 0, qi = 0, act = 0, gx = 0, ga = 0, y = 0, rl = 0, pairs = 0, ex = 0, nb = 0;
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        o = std::max(o, (size_t)T * lb_round_up(hv_of(s), 8));
        io = std::max(io, lb_img_bytes(T, hv_of(s), dt));
        if (s.mixer == LOOM_B200_MIXER_GLA) {
            const size_t C = lb_gla_chunk(s.dim, s.rank), n = lb_ceil_div(T, (int)C);
            qd = std::max(qd, (size_t)T * s.heads * s.dim);
            cs = std::max(cs, n * s.heads * s.dim * s.vdim);
            cd = std::max(cd, n * s.heads * s.dim);
            cw = std::max(cw, n * s.heads * C * C);
        } else {
            hr = std::max(hr, (size_t)std::min(T, kLatentStepTokens) * s.heads * s.rank);
            LbLatent a = latent_of(st, l, nullptr, 0);
            qi = std::max(qi, lb_latent_heads_bytes(a, T));
        }
        if (s.ffn == LOOM_B200_FFN_DENSE) act = std::max(act, lb_img_bytes(T, s.ff, dt));
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
    LB_A(pf_qd, qd * 4);
    LB_A(pf_kd, qd * 4);
    LB_A(pf_cw, cw * 4);
    LB_A(pf_part, latent_part_elems(ctx, st, std::min(T, kLatentStepTokens)) * 4);
    if (is_bf16(st)) LB_A(pf_qi, qi);
    LB_A(pf_cs, cs * 4);
    LB_A(pf_cd, cd * 4);
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
    if (int rc = lb_embed_norm(ctx, dt, st->table, d.vocab, W, st->pf_tok, T, st->scal, eps, st->pf_x, st->ldx)) return rc;
    for (auto& l : st->layers) {
        const loom_b200_layer_spec& s = l.s;
        LbNormBlock n;
        n.x = st->pf_x;
        n.ldx = st->ldx;
        n.T = T;
        n.width = W;
        n.slices = slices;
        n.gain = l.scal;
        n.eps = eps;
        n.img = st->pf_h;
        if (l.conv_w) {
            n.conv_w = l.conv_w;
            n.taps = d.conv_taps;
            n.ring_ld = st->ldx;
            n.ring = l.conv_ring + (size_t)lane * d.conv_taps * st->ldx;
            n.pos0 = pos0;
        }
        if (int rc = lb_norm_block(ctx, dt, n)) return rc;
        if (l.conv_w)
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
        if (s.mixer == LOOM_B200_MIXER_GLA) {
            LbGla a = gla_of(l, st->pf_proj, st->ldp, st->pf_o, ldo, lane);
            LbGlaBlock b;
            b.qd = st->pf_qd;
            b.kd = st->pf_kd;
            b.decay = st->pf_cd;
            b.weights = st->pf_cw;
            b.states = st->pf_cs;
            if (int rc = lb_gla_block(ctx, a, b, T, pos0)) return rc;
            if (int rc = lb_gated_heads_image(ctx, dt, st->pf_o, ldo, st->pf_proj + 2 * s.heads * s.dim + hv, st->ldp, T, s.heads, s.vdim, l.mixer_norm, eps,
                                              oslices, st->pf_io))
                return rc;
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
        if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_RESID, g)) return rc;

        if (s.ffn == LOOM_B200_FFN_NONE) continue;
        n.conv_w = nullptr;
        n.taps = 1;
        n.gain = l.scal + 1;
        if (int rc = lb_norm_block(ctx, dt, n)) return rc;
        g = LbDenseGemm();
        g.x = st->pf_h;
        g.tokens = T;
        g.slices = slices;
        if (s.ffn == LOOM_B200_FFN_DENSE) {
            g.w = l.w.up->data;
            g.rows = s.ff;
            g.img = st->pf_act;
            g.img_slices = l.w.down->slices;
            if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_GELU, g)) return rc;
            g = LbDenseGemm();
            g.x = st->pf_act;
            g.tokens = T;
            g.w = l.w.down->data;
            g.rows = W;
            g.slices = l.w.down->slices;
            g.out = st->pf_x;
            g.ldo = st->ldx;
            g.mult = mult;
            if (int rc = lb_dense_gemm(ctx, dt, LB_DEPI_RESID, g)) return rc;
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
    h.gain = st->scal + 1;
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
    b.gain = st->scal + 1;
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
