// layernorm_plan.cuh -- host side of the LAYERNORM block of layered plans (included by layered_plan.cuh): pre-norm layers
// x += mixer(LN(x; norm1)), x += ff(LN(x; norm2)) with layer norms that carry a weight and no bias, over an embedding that may add a
// hashed bigram row and a sinusoidal position vector.  Per layer the mixer is a (sliding-window) latent attention, optionally with low-rank
// queries, a learned sink and a gate per head, or a matrix memory with exponential gates (mLSTM); the feed-forward is dense gated or a
// mixture of experts weighted by the softmax over the chosen logits.
//
// Kernel sequence of one layer (decode: one row in the CUDA graph; prefill: n rows per launch):
//   row kernel (x += previous sublayer; LN)                                                 (k_block_norm_rows)
//   -> latent attention: fused query latent | latent | gate projection -> latent norms + cache write -> W_uq -> ... (ly_enqueue_latent)
//      matrix memory:    fused q | k | v | g | i | f projection -> recurrence -> per-head norm, weight, sigmoid gate
//   -> output projection -> row kernel (x += mixer; LN) -> gate/up, down or router -> experts.
// The next row kernel adds the feed-forward (the weighted sum of the chosen experts' rows) to the residual.
//
// State per layer run: the ring of latents of a latent-attention layer (position j in slot j % ring, window - 1 + chunk rows slots), or the
// matrix memory; per plan the token of every position (the bigram of a call's first token needs the one before).
#pragma once

// Validation of one LAYERNORM layer and the sizes derived from it.
static int ly_layernorm_sizes(b200_plan *p, int l, LyLayer &L, const b200_layer_spec *specs) {
    Layered &Y = *p->ly;
    b200_layer_spec &s = L.s;
    const int E = Y.c.width;
    int rc;
    if (s.mixer == B200_MIXER_LATENT_ATTENTION) {
        if (s.window <= 0) return fail(p, B200_ERR_BAD_ARG, "layer %d: window %d", l, s.window);
        if (s.sink < 0 || s.sink > 2 || s.gate < 0 || s.gate > 2) return fail(p, B200_ERR_BAD_ARG, "layer %d: sink %d / gate %d", l, s.sink, s.gate);
        if (s.kv_from >= 0 && s.kv_from < l && specs[s.kv_from].window != s.window)
            return fail(p, B200_ERR_UNSUPPORTED, "layer %d and layer %d share a cache with different windows", l, s.kv_from);
        if ((rc = ly_latent_sizes(p, l, L, Y.c.n_layers, specs))) return rc;
        ly_latent_buffers(Y, L);
    } else if (s.mixer == B200_MIXER_MLSTM) {
        if (s.heads <= 0 || s.key_dim <= 0 || s.value_dim <= 0 || !(s.gate_cap > 0.0f))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: heads %d / key %d / value %d / gate cap %g", l, s.heads, s.key_dim, s.value_dim, (double)s.gate_cap);
        s.window = 1;
        L.qd = L.kd = s.heads * s.key_dim; L.vd = L.gd = L.gr = s.heads * s.value_dim;
        L.g_off = 2 * L.qd + L.vd;
        L.Pn = 2 * L.qd + 2 * L.vd + 2 * s.heads;
        L.P = E % 64 == 0 ? (L.Pn + 127) / 128 * 128 : L.Pn; // whole tcgen05 tiles; the decode step streams Pn rows
        if (L.P > Y.maxP) Y.maxP = L.P;
        if (L.gd > Y.maxO) Y.maxO = L.gd;
        if (L.gd + s.heads > Y.maxDO) Y.maxDO = L.gd + s.heads; // read-outs and their denominators
    } else return fail(p, B200_ERR_UNSUPPORTED, "layer %d: mixer %d in a layer-norm block", l, s.mixer);
    if (s.ff_kind == B200_FF_DENSE_GATED) {
        if (s.ff_dim <= 0 || (s.ff_act != B200_ACT_GELU_TANH && s.ff_act != B200_ACT_SILU && s.ff_act != B200_ACT_RELU))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: feed-forward width %d / activation %d", l, s.ff_dim, s.ff_act);
    } else if (s.ff_kind == B200_FF_MOE) {
        if (s.moe_router != B200_MOE_SOFTMAX_CHOSEN || s.moe_identity || s.moe_shared_ff) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: router kind %d in this block", l, s.moe_router);
        if (s.ff_dim <= 0 || s.ff_experts <= 0 || s.ff_top <= 0 || s.ff_top > s.ff_experts || (size_t)(E + 3 * s.ff_experts) * 4 > (size_t)Y.smem_max ||
            (s.moe_plain ? s.ff_act != B200_ACT_RELU2 : s.ff_act != B200_ACT_SILU && s.ff_act != B200_ACT_GELU_TANH))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: %d experts of width %d, %d chosen, activation %d", l, s.ff_experts, s.ff_dim, s.ff_top, s.ff_act);
        if (s.ff_top > Y.maxTop) Y.maxTop = s.ff_top;
        if (s.ff_experts > Y.maxExperts) Y.maxExperts = s.ff_experts;
    } else if (s.ff_kind != B200_FF_NONE) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: feed-forward kind %d in this block", l, s.ff_kind);
    if (s.ff_kind != B200_FF_NONE && s.ff_dim > Y.maxF) Y.maxF = s.ff_dim;
    return B200_OK;
}

// Bigram table, token history and position frequencies.
static int ly_layernorm_embedding(b200_plan *p, const b200_tensor *tensors, int nt) {
    Layered &Y = *p->ly;
    const b200_layered_config &c = Y.c;
    const int E = c.width;
    int rc;
    if (c.bigram_buckets > 0) {
        if ((rc = dalloc(p, &Y.bigram, (size_t)(c.bigram_buckets + 1) * E * 2))) return rc;
        if ((rc = ly_mat(p, tensors, nt, "bigram", c.bigram_buckets + 1, E, Y.bigram, 0))) return rc;
        const size_t hist = (size_t)c.context_length + Y.cap;
        if ((rc = dalloc(p, &Y.tok_hist, hist * 4))) return rc;
        CK(cudaMemset(Y.tok_hist, 0, hist * 4));
    }
    if (c.sinusoid) {
        std::vector<double> f((size_t)(E + 1) / 2);
        for (size_t i = 0; i < f.size(); i++) f[i] = pow((double)c.sinusoid_base, -2.0 * (double)i / E);
        if ((rc = dalloc(p, &Y.pos_freq, f.size() * 8))) return rc;
        CK(cudaMemcpy(Y.pos_freq, f.data(), f.size() * 8, cudaMemcpyHostToDevice));
    }
    return B200_OK;
}

// Weights of one LAYERNORM layer.
static int ly_layernorm_upload(b200_plan *p, int l, LyLayer &L, const b200_tensor *tensors, int nt) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    const int E = Y.c.width;
    const std::string pre = "l" + std::to_string(l) + ".", mx = pre + "mix.", ff = pre + "mlp.";
    int rc;
    if ((rc = ly_vec_f32(p, tensors, nt, pre + "norm1", E, &L.norm1))) return rc;
    if (s.mixer == B200_MIXER_LATENT_ATTENTION) {
        if ((rc = ly_latent_mixer_upload(p, l, L, tensors, nt))) return rc;
    } else {
        if ((rc = dalloc(p, &L.w_proj, (size_t)L.P * E * 2))) return rc;
        if (L.P > L.Pn) CK(cudaMemset(L.w_proj + (size_t)L.Pn * E, 0, (size_t)(L.P - L.Pn) * E * 2));
        const char *nm[6] = {"q", "k", "v", "g", "i", "f"};
        const int rows[6] = {L.qd, L.kd, L.vd, L.gr, s.heads, s.heads};
        for (int k = 0, off = 0; k < 6; off += rows[k++])
            if ((rc = ly_mat(p, tensors, nt, mx + nm[k], rows[k], E, L.w_proj, off))) return rc;
        if ((rc = ly_vec_f32(p, tensors, nt, mx + "i.b", s.heads, &L.i_bias))) return rc;
        if ((rc = ly_vec_f32(p, tensors, nt, mx + "f.b", s.heads, &L.f_bias))) return rc;
        if ((rc = ly_vec_f32(p, tensors, nt, mx + "norm", L.gd, &L.onorm))) return rc;
        if ((rc = dalloc(p, &L.w_o, (size_t)E * L.gd * 2))) return rc;
        if ((rc = ly_mat(p, tensors, nt, mx + "o", E, L.gd, L.w_o, 0))) return rc;
    }
    if (s.ff_kind == B200_FF_NONE) return B200_OK;
    if ((rc = ly_vec_f32(p, tensors, nt, pre + "norm2", E, &L.norm2))) return rc;
    if (s.ff_kind == B200_FF_MOE) return ly_experts_upload(p, L, ff, tensors, nt);
    const int F = s.ff_dim;
    if ((rc = dalloc(p, &L.w_gu, (size_t)2 * F * E * 2))) return rc;
    if ((rc = ly_mat(p, tensors, nt, ff + "gate", F, E, L.w_gu, 0))) return rc;
    if ((rc = ly_mat(p, tensors, nt, ff + "up", F, E, L.w_gu, F))) return rc;
    if ((rc = dalloc(p, &L.w_down, (size_t)E * F * 2))) return rc;
    return ly_mat(p, tensors, nt, ff + "down", E, F, L.w_down, 0);
}

// Matrix memory of one layer, from the projection rows in PROJ to the gated read-outs in ATT32 / ATT16.
static int ly_enqueue_mlstm(b200_plan *p, bool decode, int n, const StepState *st, const LyRun &R, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    const bool h16 = !decode && !Y.f32;
    int rc;
    ly::MlstmArgs a{};
    a.heads = s.heads; a.dk = s.key_dim; a.dv = s.value_dim;
    a.q_off = 0; a.k_off = L.qd; a.v_off = 2 * L.qd; a.i_off = L.g_off + L.gr; a.f_off = a.i_off + s.heads;
    a.i_bias = L.i_bias; a.f_bias = L.f_bias; a.cap = s.gate_cap; a.q_scale = s.score_scale;
    a.vec = s.key_dim % 4 == 0 && Y.maxP % 4 == 0;
    const dim3 grid(s.heads, ly::mlstm_tiles(s.key_dim, s.value_dim)), block(MLSTM_THREADS);
    const float *P = Y.PROJ;
    switch (ly::mlstm_reg_rows(s.key_dim)) {
    case 1: rc = launch_k(p, false, ly::k_mlstm_scan<1>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 2: rc = launch_k(p, false, ly::k_mlstm_scan<2>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 4: rc = launch_k(p, false, ly::k_mlstm_scan<4>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 8: rc = launch_k(p, false, ly::k_mlstm_scan<8>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 16: rc = launch_k(p, false, ly::k_mlstm_scan<16>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 32: rc = launch_k(p, false, ly::k_mlstm_scan<32>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    default: rc = launch_k(p, false, ly::k_mlstm_scan_any, grid, dim3(256), (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO);
    }
    if (rc) return rc;
    const ly::HeadNormArgs ha{L.onorm, s.value_dim, 1, Y.DO + L.gd, s.heads, s.value_dim, Y.c.norm_eps};
    *nl += 2;
    // one row: eight heads per CTA, a warp each; a chunk has CTAs enough with one per row
    return launch_k(p, false, ly::k_head_norm_gate, dim3(n, decode ? (s.heads + 7) / 8 : 1), dim3(256), (size_t)0, (const float *)Y.DO, Y.maxDO, (const float *)(Y.PROJ + L.g_off), Y.maxP, ha,
                    h16 ? (float *)nullptr : Y.ATT32, h16 ? Y.ATT16 : (ly::bf16 *)nullptr, L.gd);
}

static int ly_enqueue_layernorm(b200_plan *p, bool decode, int n, const StepState *st, const int *tokens, bool with_head, float *trace, int *launches) {
    Layered &Y = *p->ly;
    const int E = Y.c.width;
    const bool h16 = !decode && !Y.f32; // prefill in BF16 mode rounds GEMM operands to BF16
    int nl = 0, rc;
    // what the next row kernel adds to the residual: a plain row, or the chosen experts' rows with their weights
    const float *pend_a = nullptr, *pend_b = nullptr;
    const int *pend_map = nullptr;
    int pend_terms = 0;
    float *pend_trace = nullptr;
    auto row = [&](bool embed, const float *w) {
        ly::BlockNormArgs a = ly_block_norm_args(Y);
        a.emb = embed ? Y.emb : nullptr; a.tokens = tokens; a.st = st; a.add_mult = 1.0f;
        if (embed) {
            a.bigram = Y.bigram; a.bg_buckets = Y.c.bigram_buckets; a.bg_prev = Y.c.bigram_mul_prev; a.bg_cur = Y.c.bigram_mul_cur; a.tok_hist = Y.tok_hist;
            a.pos_freq = Y.pos_freq;
        }
        a.add_a = pend_a; a.add_b = pend_b; a.add_b_terms = pend_terms; a.add_b_map = pend_map; a.add_b_wts = pend_b ? Y.moe_wts : nullptr;
        a.trace = pend_trace; a.w1 = w;
        if (w) { a.out1_32 = h16 ? nullptr : Y.A32; a.out1_16 = h16 ? Y.A16 : nullptr; }
        pend_a = pend_b = nullptr; pend_map = nullptr; pend_terms = 0; pend_trace = nullptr;
        nl++;
        return ly_launch_block_norm(p, n, a);
    };
    for (size_t r = 0; r < Y.runs.size(); r++) {
        const LyRun &R = Y.runs[r];
        const LyLayer &L = Y.layers[R.layer];
        const b200_layer_spec &s = L.s;
        if ((rc = row(r == 0, L.norm1))) return rc;
        LyTc t_proj, t_o, t_gu, t_down;
        if (Y.tc && !decode) {
            if (L.tc_proj) { t_proj.a = &Y.m_a; t_proj.b = &L.m_proj; t_proj.c = &Y.m_proj_c; }
            if (L.tc_o) { t_o.a = &L.m_att; t_o.b = &L.m_o; t_o.c = &Y.m_y_c; }
            if (L.tc_gu) { t_gu.a = &Y.m_a; t_gu.b = &L.m_gate; t_gu.b2 = &L.m_up; t_gu.c = &Y.m_y_c; }
            if (L.tc_down) { t_down.a = &L.m_h; t_down.b = &L.m_down; t_down.c = &Y.m_y_c; }
        }
        if ((rc = ly_project<ly::EPI_STORE>(p, decode, n, Y.A32, Y.A16, L.w_proj, nullptr, decode ? L.Pn : L.P, E, Y.PROJ, nullptr, Y.maxP, 0, &t_proj))) return rc;
        nl++;
        if (s.mixer == B200_MIXER_MLSTM) rc = ly_enqueue_mlstm(p, decode, n, st, R, L, &nl);
        else rc = ly_enqueue_latent(p, decode, n, st, R, L, &nl);
        if (rc) return rc;
        if ((rc = ly_project<ly::EPI_STORE>(p, decode, n, Y.ATT32, Y.ATT16, L.w_o, nullptr, E, L.gd, Y.Y, nullptr, E, 0, &t_o))) return rc;
        nl++;
        pend_a = Y.Y;
        if (s.ff_kind != B200_FF_NONE && (rc = row(false, L.norm2))) return rc;
        if (s.ff_kind == B200_FF_DENSE_GATED) {
            const int F = s.ff_dim;
            if ((rc = ly_project<ly::EPI_GATED>(p, decode, n, Y.A32, Y.A16, L.w_gu, nullptr, F, E, Y.H32, h16 ? Y.H16 : nullptr, F, s.ff_act, &t_gu))) return rc;
            if ((rc = ly_project<ly::EPI_STORE>(p, decode, n, Y.H32, Y.H16, L.w_down, nullptr, E, F, Y.Y, nullptr, E, 0, &t_down))) return rc;
            nl += 2;
            pend_a = Y.Y;
        } else if (s.ff_kind == B200_FF_MOE) {
            const ly::RouteMode rm{2, nullptr, s.ff_experts, 1.0f, L.router_b};
            if ((rc = ly_enqueue_route(p, decode, n, L, Y.A32, Y.A16, s.ff_experts, 0, rm, &nl))) return rc;
            if ((rc = ly_enqueue_experts(p, decode, n, L, Y.A32, Y.A16, s.ff_experts, false, &pend_b, &pend_map, &nl))) return rc;
            pend_terms = s.ff_top;
        }
        pend_trace = trace ? trace + r * (size_t)Y.cap * E : nullptr;
    }
    if (decode) {
        if ((rc = row(false, with_head ? Y.final_norm : nullptr))) return rc;
        if (with_head) {
            if ((rc = ly_project<ly::EPI_STORE>(p, true, 1, Y.A32, nullptr, Y.head, nullptr, Y.c.vocab_size, E, p->logits, nullptr, Y.c.vocab_size, 0))) return rc;
            nl++;
            if (Y.c.logit_softcap > 0.0f) {
                if ((rc = launch_k(p, false, ly::k_softcap, dim3((Y.c.vocab_size + 255) / 256), dim3(256), (size_t)0, p->logits, (long long)Y.c.vocab_size, Y.c.logit_softcap))) return rc;
                nl++;
            }
        }
        if ((rc = launch_k(p, false, k_argmax_advance, dim3(1), dim3(1024), (size_t)0, (const float *)p->logits, Y.c.vocab_size, p->st, (const int *)p->seq_tokens,
                           p->out_ids, with_head ? 1 : 0, (const float *)nullptr, (const int *)nullptr, 0, TraceBuf{nullptr, 0, 0}, p->tp, -1))) return rc;
        nl++;
    } else if ((rc = row(false, nullptr))) return rc;
    if (launches) *launches = nl;
    return B200_OK;
}
