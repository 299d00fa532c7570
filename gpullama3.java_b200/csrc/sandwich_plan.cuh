// sandwich_plan.cuh -- host side of what sandwich-normed layers (B200_BLOCK_SANDWICH, layered_plan.cuh) offer beside windowed attention and a
// gated feed-forward (included by layered_plan.cuh): two further mixers, two further feed-forwards and the per-layer token input.
//
//   lightning:       fused q | k | v | g projection -> decayed linear attention (k_lightning_scan; chunks of BF16 plans: k_lightning_chunk) -> one norm over
//                     all heads, sigmoid gate -> output projection
//   attention + scan: ONE fused projection q | k | v | g | x | z of both branches; then, on two streams,
//                       whole-projection q/k norm + rotation + ring write -> chunk-masked attention (+ gate, * branch_scale[0])
//                       convolution + SiLU -> W_x -> [W_dt] -> selective scan (+ gate silu(z), * branch_scale[1])
//                     write side by side into one row, which ONE output projection with the matrices [W_o left | W_o right] reduces: the branches'
//                     sum needs no pass of its own
//   plain feed-forward: up with the activation in the epilogue, down;   mixture of experts: router, selection, grouped experts (latent_plan.cuh), whose
//                     weighted sum the next row kernel assembles in front of its post-norm
//   token input:     row kernel (finishes the feed-forward) -> gate projection with gelu * (token's row) in the epilogue -> up-projection; the next row kernel
//                     norms and adds it
//
// State per layer run: the attention's ring (position j in slot j % ring), the recurrent state (FP32) and the ring of convolution inputs.
#pragma once

// Validation of a sandwich layer's feed-forward and the sizes derived from it.
static int ly_sandwich_ff_sizes(b200_plan *p, int l, const b200_layer_spec &s) {
    Layered &Y = *p->ly;
    const int E = Y.c.width;
    if (s.ff_kind == B200_FF_NONE) return B200_OK;
    if (s.ff_kind == B200_FF_DENSE_GATED) {
        if (s.ff_dim <= 0 || (s.ff_act != B200_ACT_GELU_TANH && s.ff_act != B200_ACT_SILU && s.ff_act != B200_ACT_RELU))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: feed-forward width %d / activation %d", l, s.ff_dim, s.ff_act);
    } else if (s.ff_kind == B200_FF_DENSE_PLAIN) {
        if (s.ff_dim <= 0 || s.ff_act < 0 || s.ff_act > B200_ACT_RELU2) return fail(p, B200_ERR_BAD_ARG, "layer %d: feed-forward width %d / activation %d", l, s.ff_dim, s.ff_act);
    } else if (s.ff_kind == B200_FF_MOE) {
        if (s.moe_router != B200_MOE_SOFTMAX_GROUPS || s.moe_identity || s.moe_shared_ff || s.moe_plain) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: router kind %d in this block", l, s.moe_router);
        if (s.ff_dim <= 0 || s.ff_experts <= 0 || s.ff_top <= 0 || s.ff_top > s.ff_experts || (size_t)(E + 3 * s.ff_experts) * 4 > (size_t)Y.smem_max || (size_t)3 * s.ff_experts * 4 > 49152 ||
            (s.ff_act != B200_ACT_SILU && s.ff_act != B200_ACT_GELU_TANH))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: %d experts of width %d, %d chosen, activation %d", l, s.ff_experts, s.ff_dim, s.ff_top, s.ff_act);
        if (s.moe_groups <= 0 || s.ff_experts % s.moe_groups || s.moe_keep <= 0 || s.moe_keep > s.moe_groups || s.ff_top > s.moe_keep * (s.ff_experts / s.moe_groups))
            return fail(p, B200_ERR_BAD_ARG, "layer %d: %d experts in %d groups, %d kept, %d chosen", l, s.ff_experts, s.moe_groups, s.moe_keep, s.ff_top);
        if (s.ff_top > Y.maxTop) Y.maxTop = s.ff_top;
        if (s.ff_experts > Y.maxExperts) Y.maxExperts = s.ff_experts;
    } else return fail(p, B200_ERR_UNSUPPORTED, "layer %d: feed-forward kind %d in this block", l, s.ff_kind);
    if (s.ff_dim > Y.maxF) Y.maxF = s.ff_dim;
    return B200_OK;
}

// Validation of a lightning or attention + scan mixer and the sizes derived from it.
static int ly_sandwich_mixer_sizes(b200_plan *p, int l, LyLayer &L) {
    Layered &Y = *p->ly;
    b200_layer_spec &s = L.s;
    const int E = Y.c.width;
    const bool pad = !Y.f32 && E % 64 == 0; // zero rows up to whole 128-row tiles for the tcgen05 GEMM; the decode step streams Pn rows
    if (s.heads <= 0 || s.kv_heads <= 0 || s.heads % s.kv_heads || s.key_dim <= 0 || s.value_dim <= 0 || s.window <= 0)
        return fail(p, B200_ERR_BAD_ARG, "layer %d: heads %d / kv heads %d / key %d / value %d / window %d", l, s.heads, s.kv_heads, s.key_dim, s.value_dim, s.window);
    if (s.mixer == B200_MIXER_LIGHTNING) {
        if (!ly::lightning_reg_rows(s.key_dim)) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: a state of %d rows per column exceeds the 512 the recurrence keeps in registers", l, s.key_dim);
        s.window = 1;
        L.qd = L.kd = s.heads * s.key_dim; L.vd = L.gd = L.gr = s.heads * s.value_dim;
        L.Pn = 2 * L.qd + 2 * L.vd;
        if ((size_t)L.gd * 4 > (size_t)Y.smem_max) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: a read-out row of %d values exceeds the shared memory of a CTA", l, L.gd);
        if (L.gd > Y.maxDO) Y.maxDO = L.gd;
        L.chunkwise = !Y.f32 && Y.cap > 1 && (s.key_dim == 32 || s.key_dim == 64 || s.key_dim == 128) && s.value_dim % 8 == 0;
        if (L.chunkwise && 2 * L.qd + L.vd > Y.maxLQ) Y.maxLQ = 2 * L.qd + L.vd;
    } else { // B200_MIXER_ATTENTION_SCAN
        if (s.sink || s.gate > 1 || s.qkv_bias || s.bias_rows || s.value_from_key || s.head_temp || s.head_mix)
            return fail(p, B200_ERR_UNSUPPORTED, "layer %d: sinks, per-head gates, biases, distance tables, key-values, head temperature and head mixing are not combined with a scan", l);
        if (s.rope_dims < 0 || s.rope_dims % 2 || s.rope_dims > s.key_dim || (s.rope_dims > 0 && !(s.rope_base > 0.0f)) || s.yarn_factor != 0.0f || s.rope_factor < 0.0f)
            return fail(p, B200_ERR_BAD_ARG, "layer %d: rotation of %d of %d entries, base %g", l, s.rope_dims, s.key_dim, (double)s.rope_base);
        if (s.scan_inner <= 0 || s.scan_state <= 0 || s.scan_rank <= 0 || s.conv_taps < 1 || s.conv_taps > 64)
            return fail(p, B200_ERR_BAD_ARG, "layer %d: scan of %d channels, %d states, step rank %d, %d convolution taps", l, s.scan_inner, s.scan_state, s.scan_rank, s.conv_taps);
        if (!ly::sel_reg_rows(s.scan_state)) return fail(p, B200_ERR_UNSUPPORTED, "layer %d: %d states per channel exceed the 512 the recurrence keeps in registers", l, s.scan_state);
        L.qd = s.heads * s.key_dim; L.kd = s.kv_heads * s.key_dim; L.vd = L.pv = s.kv_heads * s.value_dim;
        L.ad = s.heads * s.value_dim;
        L.gr = s.gate ? L.ad : 0;
        L.gd = L.ad + s.scan_inner;
        L.x_off = L.qd + L.kd + L.vd + L.gr;
        L.dC = s.scan_inner;
        L.Pn = L.x_off + 2 * s.scan_inner;
        L.nx = s.scan_rank + 2 * s.scan_state;
        L.nxp = !Y.f32 && s.scan_inner % 64 == 0 ? (L.nx + 127) / 128 * 128 : (L.nx + 3) / 4 * 4;
        if (L.nxp > Y.maxX) Y.maxX = L.nxp;
        if (s.scan_rank > Y.maxRank) Y.maxRank = s.scan_rank;
        if ((s.scan_inner + 7) / 8 * 8 > Y.maxD) Y.maxD = (s.scan_inner + 7) / 8 * 8;
        if ((s.scan_inner + 3) / 4 * 4 > Y.maxQ) Y.maxQ = (s.scan_inner + 3) / 4 * 4;
        if (s.conv_taps > Y.max_taps) Y.max_taps = s.conv_taps;
        if (s.window > Y.max_window) Y.max_window = s.window;
        if (s.value_dim > Y.max_att_dv) Y.max_att_dv = s.value_dim;
    }
    L.P = pad ? (L.Pn + 127) / 128 * 128 : L.Pn;
    if (L.P > Y.maxP) Y.maxP = L.P;
    if (L.gd > Y.maxO) Y.maxO = L.gd;
    return B200_OK;
}

// rows x cols BF16 matrix into columns [col_off, col_off + cols) of dst [rows][ld]
static int ly_mat_cols(b200_plan *p, const b200_tensor *tensors, int nt, const std::string &name, int rows, int cols, ly::bf16 *dst, int ld, int col_off) {
    const b200_tensor *t = find(tensors, nt, name);
    if (!t) return fail(p, B200_ERR_BAD_ARG, "missing tensor %s", name.c_str());
    if (t->ggml_type != B200_GGML_BF16 || t->n_dims != 2 || t->dims[0] != cols || t->dims[1] != rows) return fail(p, B200_ERR_BAD_ARG, "tensor %s is not BF16 [%d][%d]", name.c_str(), rows, cols);
    CK(cudaMemcpy2D(dst + col_off, (size_t)ld * 2, t->data, (size_t)cols * 2, (size_t)cols * 2, rows, cudaMemcpyHostToDevice));
    p->up.h2d_bytes += (int64_t)rows * cols * 2;
    return B200_OK;
}

static int ly_sandwich_mixer_upload(b200_plan *p, int l, LyLayer &L, const b200_tensor *tensors, int nt) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    const int E = Y.c.width;
    const std::string mx = "l" + std::to_string(l) + ".mix.";
    int rc;
    if ((rc = dalloc(p, &L.w_proj, (size_t)L.P * E * 2))) return rc;
    if (L.P > L.Pn) CK(cudaMemset(L.w_proj + (size_t)L.Pn * E, 0, (size_t)(L.P - L.Pn) * E * 2));
    if ((rc = dalloc(p, &L.w_o, (size_t)E * L.gd * 2))) return rc;
    const bool light = s.mixer == B200_MIXER_LIGHTNING;
    const std::string at = light ? mx : mx + "left.";
    const char *nm[4] = {"q", "k", "v", "g"};
    const int rows[4] = {L.qd, L.kd, L.vd, L.gr};
    for (int k = 0, off = 0; k < 4; off += rows[k++])
        if (rows[k] > 0 && (rc = ly_mat(p, tensors, nt, at + nm[k], rows[k], E, L.w_proj, off))) return rc;
    if (light) {
        if ((rc = ly_vec_f32(p, tensors, nt, mx + "decay", s.heads, &L.decay))) return rc;
        if ((rc = ly_vec_f32(p, tensors, nt, mx + "norm", L.gd, &L.onorm))) return rc;
        return ly_mat(p, tensors, nt, mx + "o", E, L.gd, L.w_o, 0);
    }
    if (s.qk_norm) {
        if ((rc = ly_vec_f32(p, tensors, nt, at + "q.norm", L.qd, &L.qnorm))) return rc;
        if ((rc = ly_vec_f32(p, tensors, nt, at + "k.norm", L.kd, &L.knorm))) return rc;
    }
    if (s.rope_dims > 0 && (rc = ly_rope_table(p, s, Y.c.context_length, &L.rope))) return rc;
    const std::string sc = mx + "right.";
    const int I = s.scan_inner, N = s.scan_state;
    if ((rc = ly_mat(p, tensors, nt, sc + "in", 2 * I, E, L.w_proj, L.x_off))) return rc;
    if ((rc = ly_mat_cols(p, tensors, nt, at + "o", E, L.ad, L.w_o, L.gd, 0))) return rc;
    if ((rc = ly_mat_cols(p, tensors, nt, sc + "o", E, I, L.w_o, L.gd, L.ad))) return rc;
    if ((rc = ly_vec_f32(p, tensors, nt, sc + "conv", (int64_t)I * s.conv_taps, &L.conv_w))) return rc;
    if ((rc = ly_vec_f32(p, tensors, nt, sc + "conv.b", I, &L.conv_b))) return rc;
    if ((rc = dalloc(p, &L.w_x, (size_t)L.nxp * I * 2))) return rc;
    CK(cudaMemset(L.w_x, 0, (size_t)L.nxp * I * 2));
    if ((rc = ly_mat(p, tensors, nt, sc + "x", L.nx, I, L.w_x, 0))) return rc;
    if ((rc = dalloc(p, &L.w_dt, (size_t)I * s.scan_rank * 2))) return rc;
    if ((rc = ly_mat(p, tensors, nt, sc + "dt", I, s.scan_rank, L.w_dt, 0))) return rc;
    if ((rc = ly_vec_f32(p, tensors, nt, sc + "dt.b", I, &L.dt_bias))) return rc;
    if ((rc = ly_vec_f32(p, tensors, nt, sc + "D", I, &L.ssd_d))) return rc;
    // decay exponents in base 2, evaluated in double: S <- 2^(a2 dt) S
    std::vector<float> a;
    if ((rc = ly_bf16_host(p, tensors, nt, sc + "A_log", (int64_t)I * N, a))) return rc;
    for (float &v : a) v = (float)(-exp((double)v) * 1.4426950408889634074);
    if ((rc = dalloc(p, &L.a2, a.size() * 4))) return rc;
    CK(cudaMemcpy(L.a2, a.data(), a.size() * 4, cudaMemcpyHostToDevice));
    return B200_OK;
}

// Plain feed-forward or mixture of experts of a sandwich layer (norms: the caller).
static int ly_sandwich_ff_upload(b200_plan *p, int l, LyLayer &L, const b200_tensor *tensors, int nt) {
    const b200_layer_spec &s = L.s;
    const int E = p->ly->c.width, F = s.ff_dim;
    const std::string ff = "l" + std::to_string(l) + ".mlp.";
    if (s.ff_kind == B200_FF_MOE) return ly_experts_upload(p, L, ff, tensors, nt);
    int rc;
    if ((rc = dalloc(p, &L.w_gu, (size_t)F * E * 2))) return rc;
    if ((rc = ly_mat(p, tensors, nt, ff + "up", F, E, L.w_gu, 0))) return rc;
    if ((rc = dalloc(p, &L.w_down, (size_t)E * F * 2))) return rc;
    return ly_mat(p, tensors, nt, ff + "down", E, F, L.w_down, 0);
}

// Per-layer token input: gate rows padded with zeros to whole tcgen05 tiles.
static int ly_side_upload(b200_plan *p, int l, LyLayer &L, const b200_tensor *tensors, int nt) {
    Layered &Y = *p->ly;
    const int E = Y.c.width, D = Y.c.side_dim;
    const std::string sd = "l" + std::to_string(l) + ".side.";
    int rc;
    if ((rc = dalloc(p, &L.w_sgate, (size_t)Y.side_pad * E * 2))) return rc;
    CK(cudaMemset(L.w_sgate, 0, (size_t)Y.side_pad * E * 2));
    if ((rc = ly_mat(p, tensors, nt, sd + "gate", D, E, L.w_sgate, 0))) return rc;
    if ((rc = dalloc(p, &L.w_sproj, (size_t)E * D * 2))) return rc;
    if ((rc = ly_mat(p, tensors, nt, sd + "proj", E, D, L.w_sproj, 0))) return rc;
    return ly_vec_f32(p, tensors, nt, sd + "norm", E, &L.side_norm);
}

// State of a run with one of the two mixers (the attention's rings: the caller).
static int ly_sandwich_run(b200_plan *p, LyRun &R, const LyLayer &L) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    int rc;
    if (s.mixer == B200_MIXER_LIGHTNING) R.s_floats = ly::lightning_state_floats(s.heads, s.key_dim, s.value_dim);
    else {
        R.s_floats = ly::sel_state_floats(s.scan_inner, s.scan_state);
        R.c_floats = (size_t)Y.cring * L.dC;
        if ((rc = dalloc(p, &R.cstate, R.c_floats * 4))) return rc;
        CK(cudaMemset(R.cstate, 0, R.c_floats * 4));
    }
    if ((rc = dalloc(p, &R.S, R.s_floats * 4))) return rc;
    CK(cudaMemset(R.S, 0, R.s_floats * 4));
    return B200_OK;
}

// TMA descriptors of the scan's products, the plain feed-forward and the token input (fused and output projections: the common ones).
static void ly_sandwich_tc_init(b200_plan *p) {
    Layered &Y = *p->ly;
    const int E = Y.c.width, D = Y.c.side_dim;
    const uint64_t rows = (uint64_t)Y.cap_pad;
    auto fits = [](int N, int K) { return N % 128 == 0 && K % 64 == 0; };
    const bool xp_c = Y.XP && Y.maxX % 4 == 0 && pg::make_map_c(&Y.m_xp_c, Y.XP, rows, Y.maxX) == 0;
    const bool dt_c = Y.Q && Y.maxQ % 4 == 0 && pg::make_map_c(&Y.m_dt_c, Y.Q, rows, Y.maxQ) == 0;
    const bool side_a = D > 0 && D % 64 == 0 && pg::make_map(&Y.m_side, Y.SIDE16, rows, D, pg::BM) == 0 && pg::make_map_c(&Y.m_sidef_c, Y.SIDEF, rows, Y.side_pad) == 0;
    for (LyLayer &L : Y.layers) {
        const b200_layer_spec &s = L.s;
        if (s.mixer == B200_MIXER_ATTENTION_SCAN) {
            const int I = s.scan_inner, Rk = s.scan_rank;
            L.tc_wx = xp_c && fits(L.nxp, I) && pg::make_map(&L.m_wx, L.w_x, L.nxp, I, 128) == 0 && pg::make_map_ld(&L.m_u, Y.U16, rows, I, Y.maxD, pg::BM) == 0;
            L.tc_wdt = dt_c && fits(I, Rk) && pg::make_map(&L.m_wdt, L.w_dt, I, Rk, 128) == 0 && pg::make_map(&L.m_dt16, Y.DT16, rows, Rk, pg::BM) == 0;
        }
        if (s.ff_kind == B200_FF_DENSE_PLAIN) {
            const int F = s.ff_dim;
            L.tc_gu = fits(F, E) && (s.ff_act == B200_ACT_RELU2) && pg::make_map(&L.m_up, L.w_gu, F, E, 128) == 0;
            L.tc_down = fits(E, F) && pg::make_map(&L.m_down, L.w_down, E, F, 128) == 0 && pg::make_map(&L.m_h, Y.H16, rows, F, pg::BM) == 0;
        }
        L.tc_side = side_a && fits(Y.side_pad, E) && fits(E, D) && pg::make_map(&L.m_tsg, L.w_sgate, Y.side_pad, E, 128) == 0 && pg::make_map(&L.m_tsp, L.w_sproj, E, D, 128) == 0;
    }
}

#define LC_CHUNK_MIN 16 // rows from which a chunk takes the tensor-core form
// Decayed linear attention of one layer, from the projection rows in PROJ to the gated read-outs in ATT32 / ATT16.
static int ly_enqueue_lightning(b200_plan *p, bool decode, int n, const StepState *st, const LyRun &R, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    const bool h16 = !decode && !Y.f32;
    int rc;
    ly::LightningArgs a{};
    a.heads = s.heads; a.dk = s.key_dim; a.dv = s.value_dim; a.q_off = 0; a.k_off = L.qd; a.v_off = 2 * L.qd; a.decay = L.decay;
    const dim3 grid(s.heads, (s.value_dim + LIGHT_COLS - 1) / LIGHT_COLS), block(LIGHT_THREADS);
    const float *P = Y.PROJ;
    if (h16 && L.chunkwise && n >= LC_CHUNK_MIN) {
        const int w = 2 * L.qd + L.vd;
        if ((rc = launch_k(p, false, ly::k_act_rows, dim3(n), dim3(256), (size_t)0, P, Y.maxP, w, (int)ly::ACT_SILU, Y.LQ16, w, ly::TokenGate{}))) return rc;
        const bool wide = s.heads * ((s.value_dim + 63) / 64) >= p->n_sms;
        const int cols = wide ? 64 : 32;
        const dim3 cgrid(s.heads, (s.value_dim + cols - 1) / cols), cblock(4 * cols);
        const ly::bf16 *qkv = Y.LQ16;
#define LY_CHUNK_CASE(DK) \
        if (s.key_dim == DK) rc = wide ? launch_k(p, false, ly::k_lightning_chunk<DK, 64>, cgrid, cblock, ly::lightning_chunk_smem<DK, 64>(), qkv, w, a, R.S, n, st, Y.DO, Y.maxDO) \
                                       : launch_k(p, false, ly::k_lightning_chunk<DK, 32>, cgrid, cblock, ly::lightning_chunk_smem<DK, 32>(), qkv, w, a, R.S, n, st, Y.DO, Y.maxDO);
        LY_CHUNK_CASE(32)
        LY_CHUNK_CASE(64)
        LY_CHUNK_CASE(128)
#undef LY_CHUNK_CASE
        ++*nl;
    } else switch (ly::lightning_reg_rows(s.key_dim)) {
    case 1: rc = launch_k(p, false, ly::k_lightning_scan<1>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 2: rc = launch_k(p, false, ly::k_lightning_scan<2>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 4: rc = launch_k(p, false, ly::k_lightning_scan<4>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 8: rc = launch_k(p, false, ly::k_lightning_scan<8>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    case 16: rc = launch_k(p, false, ly::k_lightning_scan<16>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO); break;
    default: rc = launch_k(p, false, ly::k_lightning_scan<32>, grid, block, (size_t)0, P, Y.maxP, a, R.S, n, st, Y.DO, Y.maxDO);
    }
    if (rc) return rc;
    *nl += 2;
    // one statistic over all heads
    return launch_k(p, false, ly::k_gated_group_norm, dim3(n), dim3(n == 1 && L.gd >= 2048 ? 1024 : 256), (size_t)L.gd * 4, (const float *)Y.DO, Y.maxDO, (const float *)(Y.PROJ + 2 * L.qd + L.vd), Y.maxP,
                    (const float *)L.onorm, L.gd, 1, Y.c.norm_eps, 1, h16 ? (float *)nullptr : Y.ATT32, h16 ? Y.ATT16 : (ly::bf16 *)nullptr, L.gd);
}

// Selective scan of one layer, from the x and z columns of PROJ to the columns behind the attention's in ATT32 / ATT16.
static int ly_enqueue_selective(b200_plan *p, bool decode, int n, const StepState *st, const LyRun &R, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    const b200_layer_spec &s = L.s;
    const bool h16 = !decode && !Y.f32, one = n == 1;
    const int I = s.scan_inner, N = s.scan_state, Rk = s.scan_rank;
    int rc;
    ly::ConvArgs ca{};
    ca.C = I; ca.taps = s.conv_taps; ca.cring = Y.cring; ca.w = L.conv_w; ca.bias_out = L.conv_b; ca.silu = 1;
    if ((rc = launch_k(p, false, ly::k_conv_rows, dim3((n + LY_CONV_ROWS - 1) / LY_CONV_ROWS, (I + 255) / 256), dim3(256), (size_t)0, (const float *)Y.PROJ, Y.maxP, L.x_off, ca, R.cstate, Y.DLT, Y.maxD,
                       h16 ? Y.U16 : (ly::bf16 *)nullptr, Y.maxD, st, n))) return rc;
    if (h16 && Y.tc && L.tc_wx) {
        LyTc t; t.a = &L.m_u; t.b = &L.m_wx; t.c = &Y.m_xp_c;
        rc = ly_project<ly::EPI_STORE>(p, false, n, nullptr, Y.U16, L.w_x, nullptr, L.nxp, I, Y.XP, nullptr, Y.maxX, 0, &t);
    } else {
        ly::GemmView gv{};
        gv.lda = Y.maxD;
        rc = ly_project_view<ly::EPI_STORE>(p, decode, n, Y.DLT, Y.U16, L.w_x, L.nx, I, Y.XP, nullptr, Y.maxX, 0, gv, ly::MvView{}, 1, 1, 0);
    }
    if (rc) return rc;
    *nl += 3;
    if (!one) { // step sizes of the chunk; a single row's are computed inside the scan
        ly::GemmView gv{};
        if (h16) {
            if ((rc = launch_k(p, false, ly::k_act_rows, dim3(n), dim3(256), (size_t)0, (const float *)Y.XP, Y.maxX, Rk, (int)ly::ACT_NONE, Y.DT16, Rk, ly::TokenGate{}))) return rc;
            ++*nl;
        }
        ++*nl;
        if (h16 && Y.tc && L.tc_wdt) {
            LyTc t; t.a = &L.m_dt16; t.b = &L.m_wdt; t.c = &Y.m_dt_c;
            rc = ly_project<ly::EPI_STORE>(p, false, n, nullptr, Y.DT16, L.w_dt, nullptr, I, Rk, Y.Q, nullptr, Y.maxQ, 0, &t);
        } else {
            gv.lda = h16 ? Rk : Y.maxX;
            rc = ly_project_view<ly::EPI_STORE>(p, false, n, Y.XP, Y.DT16, L.w_dt, I, Rk, Y.Q, nullptr, Y.maxQ, 0, gv, ly::MvView{}, 1, 1, 0);
        }
        if (rc) return rc;
    }
    ly::SelScanArgs a{};
    a.C = I; a.N = N; a.rank = Rk; a.a2 = L.a2; a.dt_bias = L.dt_bias; a.D = L.ssd_d; a.w_dt = one ? L.w_dt : nullptr; a.out_scale = s.branch_scale[1];
    const int z_off = L.x_off + I;
    a.vec = I % 4 == 0 && N % 4 == 0 && Rk % 4 == 0 && z_off % 4 == 0 && Y.maxP % 4 == 0 && Y.maxX % 4 == 0 && Y.maxQ % 4 == 0 && Y.maxD % 4 == 0;
    const int lpc = ly::sel_lanes(N), ch = SEL_THREADS / lpc;
    const dim3 grid((I + ch - 1) / ch), block(SEL_BLOCK);
    const float *U = Y.DLT, *PX = Y.XP, *DT = Y.Q, *Z = Y.PROJ + z_off;
    float *o32 = h16 ? nullptr : Y.ATT32 + L.ad;
    ly::bf16 *o16 = h16 ? Y.ATT16 + L.ad : nullptr;
    const int rr = ly::sel_reg_rows(N);
    if (lpc > SEL_LANES) {
        if (rr == 8) return launch_k(p, false, ly::k_selective_scan<32, 8>, grid, block, ly::sel_smem(32, 8), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
        return launch_k(p, false, ly::k_selective_scan<32, 16>, grid, block, ly::sel_smem(32, 16), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    }
    switch (rr) {
    case 1: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 1>, grid, block, ly::sel_smem(SEL_LANES, 1), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    case 2: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 2>, grid, block, ly::sel_smem(SEL_LANES, 2), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    case 4: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 4>, grid, block, ly::sel_smem(SEL_LANES, 4), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    case 8: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 8>, grid, block, ly::sel_smem(SEL_LANES, 8), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    case 16: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 16>, grid, block, ly::sel_smem(SEL_LANES, 16), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    default: return launch_k(p, false, ly::k_selective_scan<SEL_LANES, 32>, grid, block, ly::sel_smem(SEL_LANES, 32), U, Y.maxD, PX, Y.maxX, DT, Y.maxQ, Z, Y.maxP, a, R.S, n, st, o32, o16, L.gd);
    }
}

// Both branches of an attention + scan mixer, the scan on a stream of its own: they read disjoint columns of the projection rows and write disjoint
// columns of the output rows.  Inside a capture the two streams become parallel branches of the graph.
static int ly_enqueue_attention_scan(b200_plan *p, bool decode, int n, const StepState *st, const LyRun &R, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    cudaStream_t main = p->stream;
    if (cudaEventRecord(Y.ev_fork, main) != cudaSuccess || cudaStreamWaitEvent(Y.branch, Y.ev_fork, 0) != cudaSuccess) return fail(p, B200_ERR_CUDA, "stream fork failed");
    p->stream = Y.branch;
    const int rs = ly_enqueue_selective(p, decode, n, st, R, L, nl);
    p->stream = main;
    const int ra = rs ? rs : ly_enqueue_attention(p, decode, n, st, R, L, nl);
    // joined also on failure: a capture must not end with an open branch
    if (cudaEventRecord(Y.ev_join, Y.branch) != cudaSuccess || cudaStreamWaitEvent(main, Y.ev_join, 0) != cudaSuccess) return ra ? ra : fail(p, B200_ERR_CUDA, "stream join failed");
    return ra;
}

// Plain feed-forward of one layer from the normed rows in A32 / A16 to Y.Y.
static int ly_enqueue_plain_ff(b200_plan *p, bool decode, int n, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    const int E = Y.c.width, F = L.s.ff_dim;
    const bool h16 = !decode && !Y.f32;
    int rc;
    if (h16 && Y.tc && L.tc_gu) { // activation and rounding in the epilogue of the tcgen05 GEMM
        const uint32_t fl = pg::FLAVOR_BF16 | pg::FLAVOR_RELU2_BF16;
        const int g = F % 256 == 0 ? pg::gemm2_persist_launch<pg::GEMM_ACT, 256, pg::GEMM2_PERSIST_STAGES_256>(Y.m_a, L.m_up, L.m_up, Y.m_y_c, Y.H16, F, n, (n + 255) / 256 * 2, F / 256, E, p->n_sms, p->stream, 1, fl)
                                   : pg::gemm_launch<pg::GEMM_ACT, pg::GEMM_STAGES>(Y.m_a, L.m_up, L.m_up, Y.m_y_c, Y.H16, F, n, (n + 127) / 128, F / 128, E, p->stream, fl);
        if (g) return fail(p, B200_ERR_CUDA, "tensor-core GEMM launch failed (%d)", g);
    } else if ((rc = ly_project<ly::EPI_ACT>(p, decode, n, Y.A32, Y.A16, L.w_gu, nullptr, F, E, Y.H32, h16 ? Y.H16 : nullptr, F, L.s.ff_act))) return rc;
    LyTc t;
    if (Y.tc && !decode && L.tc_down) { t.a = &L.m_h; t.b = &L.m_down; t.c = &Y.m_y_c; }
    *nl += 2;
    return ly_project<ly::EPI_STORE>(p, decode, n, Y.H32, Y.H16, L.w_down, nullptr, E, F, Y.Y, nullptr, E, 0, &t);
}

// Per-layer token input of layer l: reads the residual rows (FP32 from X, or their BF16 rounding in A16), leaves P (gelu_tanh(G x) * e) in Y.Y.
static int ly_enqueue_side(b200_plan *p, bool decode, int n, const StepState *st, const int *tokens, int l, const LyLayer &L, int *nl) {
    Layered &Y = *p->ly;
    const int E = Y.c.width, D = Y.c.side_dim;
    const bool h16 = !decode && !Y.f32;
    const ly::TokenGate tg{Y.side_emb + (size_t)l * D, Y.c.n_layers * D, decode ? nullptr : tokens, st};
    int rc;
    *nl += 2;
    if (h16 && Y.tc && L.tc_side) {
        LyTc t, t2;
        t.a = &Y.m_a; t.b = &L.m_tsg; t.c = &Y.m_sidef_c;
        if ((rc = ly_project<ly::EPI_STORE>(p, false, n, nullptr, Y.A16, L.w_sgate, nullptr, Y.side_pad, E, Y.SIDEF, nullptr, Y.side_pad, 0, &t))) return rc;
        if ((rc = launch_k(p, false, ly::k_act_rows, dim3(n), dim3(256), (size_t)0, (const float *)Y.SIDEF, Y.side_pad, D, (int)ly::ACT_GELU_TANH, Y.SIDE16, D, tg))) return rc;
        t2.a = &Y.m_side; t2.b = &L.m_tsp; t2.c = &Y.m_y_c;
        ++*nl;
        return ly_project<ly::EPI_STORE>(p, false, n, nullptr, Y.SIDE16, L.w_sproj, nullptr, E, D, Y.Y, nullptr, E, 0, &t2);
    }
    ly::GemmView gv{};
    ly::MvView mv{};
    gv.tg = mv.tg = tg;
    if ((rc = ly_project_view<ly::EPI_ACT>(p, decode, n, Y.X, Y.A16, L.w_sgate, D, E, Y.SIDE32, h16 ? Y.SIDE16 : nullptr, D, B200_ACT_GELU_TANH, gv, mv, 1, 1, 0))) return rc;
    return ly_project<ly::EPI_STORE>(p, decode, n, Y.SIDE32, Y.SIDE16, L.w_sproj, nullptr, E, D, Y.Y, nullptr, E, 0);
}
