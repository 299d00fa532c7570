"""GPU tests of the layer-norm block of layered plans (csrc/layernorm_plan.cuh, csrc/mlstm.cuh and the kernels it shares with the
other layered designs) on small random Kegasun models, against the float64 oracle (oracle/kegasun_oracle.py, which shares no code
with the product).

Tolerances.  FP32 compute mode and the decode step (FP32 activations in either mode): relative RMS error of a logits row
<= 5e-5 (only the summation order differs): this is the sharp comparison, and every case runs in it.  BF16 compute mode, batched
prefill: GEMM operands are rounded to BF16 and the untrained random layers pass the rounding of every layer on to the next, so the
bound grows with depth: 1.2 % per layer (+ 1 for the classifier).  In BF16 mode the routers never face a close call (see
kegasun_util.decisive_routing), and no read-out of the matrix memory is one that rounding may turn (kegasun_util.rounding_shift).  Where a test plants a key or a write that decides the output, the model has one layer (bound 2.4 %) and
a slip of the cache or the state moves the row by more than 10 %."""
import numpy as np
import pytest

from kegasun_util import bf16_values, configs, decisive_routing, min_margin, needle_attention, needle_mlstm, oracle, random_layer_list, rel_rms, rounding_shift, settled_weights, w64

pytestmark = pytest.mark.gpu

TOL_DECODE = 5e-5
ALL = ["mixed", "odd", "attention_only", "memory_only", "tiles_a", "tiles_b"]


def tol(compute, cfg):
    return 5e-5 if compute == "float32" else 1.2e-2 * (len(cfg["layers"]) + 1)


def weights_for(S, O, cfg, seed, compute, toks):
    """Random weights; in BF16 mode with decisive routers and no read-out that rounding may turn.  In FP32 mode the seed must not produce a near-tie of two experts."""
    if compute == "bfloat16":
        w = settled_weights(S, O, cfg, seed, toks, 0.5 * tol(compute, cfg))
    else:
        w = S.kegasun_weights(cfg, seed)
        assert min_margin(O, cfg, w64(w), toks) > 1e-4, "near-tie of two experts in the oracle: pick another seed"
    return w


def make_plan(pkg, cfg, weights, ctx=256, batch=16, compute="float32"):
    model = pkg.synth.kegasun_model(cfg, weights, ctx)
    return pkg.B200MasterPlan.initialize_plan(model, prefill_batch_size=batch, compute=compute)


def prefill_all(plan, toks, batch, start=0):
    rows = []
    for c0 in range(0, len(toks), batch):
        part = toks[c0:c0 + batch]
        lg, _ = plan.forward_batch_logits(part, start + c0, list(range(len(part))))
        rows.append(lg)
    return np.concatenate(rows)


def assert_rows(got, ref, bound, what=""):
    errs = [rel_rms(got[i], ref[i]) for i in range(len(ref))]
    worst = int(np.argmax(errs))
    assert errs[worst] <= bound, f"{what}: relative RMS error {errs[worst]:.3g} > {bound} at row {worst}"


def portions(plan, toks, sizes, batch):
    """The prompt in portions of the given sizes (each cut again at the chunk capacity; a portion of one token is a decode step),
    the rest decoded one by one."""
    got, p = [], 0
    for m in sizes:
        if m == 1:
            got.append(plan.forward_decode(toks[p], p)[0][None])
        else:
            got.append(prefill_all(plan, toks[p:p + m], batch, start=p))
        p += m
    while p < len(toks):
        got.append(plan.forward_decode(toks[p], p)[0][None])
        p += 1
    return np.concatenate(got)


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ALL)
def test_every_layer_matches_oracle(pkg, name, compute):
    """Residual stream after every layer and the logits: each mixer alone (memory_only, attention_only) and in every order, with and
    without feed-forwards."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(5).integers(0, cfg["vocab"], 23).tolist()
    w = weights_for(S, O, cfg, 11, compute, toks)
    ref_lg, ref_tr = O.forward(cfg, w64(w), toks, return_layers=True)
    plan = make_plan(pkg, cfg, w, batch=32, compute=compute)
    try:
        assert plan.layered_info()[0] == len(ref_tr)
        lg, tr = plan.forward_batch_logits(toks, 0, list(range(len(toks))), want_trace=True)
        for r in range(len(ref_tr)):
            assert rel_rms(tr[r], ref_tr[r]) <= tol(compute, cfg), f"layer {r}"
        assert_rows(lg, ref_lg, tol(compute, cfg), "logits")
    finally:
        plan.free()


@pytest.mark.parametrize("name", ALL)
def test_prefill_equals_token_by_token_decode(pkg, name):
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(6).integers(0, cfg["vocab"], 60).tolist()
    for compute in ("float32", "bfloat16"):
        w = weights_for(S, O, cfg, 12, compute, toks)
        ref = O.forward(cfg, w64(w), toks)
        plan = make_plan(pkg, cfg, w, batch=64, compute=compute)
        try:
            whole = prefill_all(plan, toks, 64)
            step = np.stack([plan.forward_decode(t, p)[0] for p, t in enumerate(toks)])  # position 0 starts from an empty state without a reset
            assert_rows(step, ref, TOL_DECODE, "decode")
            assert_rows(whole, ref, tol(compute, cfg), "prefill")
        finally:
            plan.free()


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "attention_only", "memory_only"])
def test_portions_of_every_size(pkg, name, compute):
    """The same prompt cut into portions of 1 .. 13 tokens (the previous token across every edge, edges inside the windows and inside
    the recurrence's batches of tokens), then decoded one by one; the chunk capacity (7) is below the portion sizes, so portions are
    cut again, and the rings have just window - 1 + 7 slots."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 70).tolist()
    w = weights_for(S, O, cfg, 13, compute, toks)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, ctx=70, batch=7, compute=compute)  # the last token fills the context
    try:
        windows = [lc["mixer"]["mask"]["size"] for lc in cfg["layers"] if lc["type"] == "latent_attention"]
        assert plan.layered_info()[1] == min(70, max([min(x, 70) for x in windows] + [1]) - 1 + 7)
        for sizes in ([2, 3, 2, 13, 5, 2, 11, 2, 7], [9, 2, 1, 2, 2, 12, 1, 1, 3], [50], [2] * 20, [1, 2, 1, 60]):
            assert_rows(portions(plan, toks, sizes, 7), ref, tol(compute, cfg), f"portions {sizes}")
    finally:
        plan.free()


@pytest.mark.parametrize("name", ["tiles_a", "tiles_b"])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_tensor_core_prefill_shapes(pkg, name, compute):
    """Shapes that take the tcgen05 GEMMs and the tensor-core attention in BF16 mode: a prompt longer than several key tiles and than
    the rings, whole, in ragged portions (of 100 rows: keys expanded per head; of a few rows behind many cached ones: the folded form),
    then decoded; then a second request over the same rings."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(12).integers(0, cfg["vocab"], 330).tolist()
    w = weights_for(S, O, cfg, 21, compute, toks)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, ctx=340, batch=100, compute=compute)
    try:
        assert_rows(prefill_all(plan, toks, 100), ref, tol(compute, cfg), "whole")
        assert_rows(portions(plan, toks, (65, 2, 100, 1, 5, 3, 90, 2, 20), 100), ref, tol(compute, cfg), "portions")
        assert_rows(prefill_all(plan, toks[:30], 100), ref[:30], tol(compute, cfg), "second request")
    finally:
        plan.free()


def test_state_and_slots_are_reused_across_requests(pkg):
    """Request after request on one plan without clearing anything: a request starts without a previous token, from an empty memory
    (and a running maximum of zero) and sees none of the earlier keys; kv_reset in between changes nothing."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)["mixed"]
    rng = np.random.default_rng(8)
    seqs = [rng.integers(0, cfg["vocab"], n).tolist() for n in (30, 3, 41, 1, 17, 2)]
    w = weights_for(S, O, cfg, 14, "float32", sum(seqs, []))
    plan = make_plan(pkg, cfg, w, ctx=48, batch=4, compute="float32")
    try:
        for k, toks in enumerate(seqs):
            n = len(toks)
            ref = O.forward(cfg, w64(w), toks)
            cut = n // 2
            got = [prefill_all(plan, toks[:cut], 4)] if cut else []
            got += [plan.forward_decode(toks[p], p)[0][None] for p in range(cut, n)]
            assert_rows(np.concatenate(got), ref, tol("float32", cfg), f"request of {n}")
            assert np.abs(plan.read_buffer("delta_state", 32, layer=1)).max() > 0
            if k == 2:
                plan.kv_reset()
                assert np.abs(plan.read_buffer("delta_state", 32, layer=1)).max() == 0
        with pytest.raises(pkg.native.B200Error):
            plan.read_buffer("conv_state", 4, layer=1)
    finally:
        plan.free()


@pytest.mark.parametrize("shape", [(8, 12), (64, 64)])
@pytest.mark.parametrize("window", [1, 2, 37, 64, 65, 150])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_window_edges_with_a_planted_key(pkg, compute, window, shape):
    """One key decides the output.  It sits at the last visible distance, one beyond it, at distances inside, at the first positions
    of the sequence, on both sides of a chunk edge and of the ring's last slot -- in a prompt (whole and in portions), with the query
    decoded after a prefill, and with everything decoded.  (64, 64): the tensor-core attention in BF16 mode."""
    S, O = pkg.synth, oracle()
    cfg, w, A, B, fill = needle_attention(S, window, *shape)
    wd = w64(w)
    ctx, batch = 330, 64
    plan = make_plan(pkg, cfg, w, ctx=ctx, batch=batch, compute=compute)
    bound = tol(compute, cfg)
    try:
        ring = plan.layered_info()[1]
        places = {(i, i - d) for i in (window, 63, 64, 65, 129, ring, ring + 1, ctx - 1) for d in (window - 1, window, 1, window // 2)} | {(window - 1, 0), (3, 0), (1, 0)}
        for i, at in sorted(places):
            if not 0 <= at < i < ctx:
                continue
            toks = [fill[(7 * t + 3) % len(fill)] for t in range(i + 1)]
            toks[i] = A
            without = O.forward(cfg, wd, toks)[i]
            toks[at] = B
            ref = O.forward(cfg, wd, toks)[i]
            if i - at < window:
                assert rel_rms(without, ref) > 0.1, "the planted key has teeth"
            assert rel_rms(prefill_all(plan, toks, batch)[i], ref) <= bound, f"prompt, query {i}, key at {at}"
            assert rel_rms(portions(plan, toks, [2] * ((i + 1) // 2) if i < 70 else [61, 2, 3, i - 66], batch)[i], ref) <= bound, f"portions, query {i}, key at {at}"
            prefill_all(plan, toks[:i], batch)
            assert rel_rms(plan.forward_decode(toks[i], i)[0], ref) <= bound, f"decoded query {i}, key at {at}"  # the keys came from the prefill kernels
            plan.decode_sequence(toks, i + 1, 0, feedback=False)
            assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref) <= TOL_DECODE, f"all decoded, query {i}, key at {at}"
    finally:
        plan.free()


@pytest.mark.parametrize("key_dim,value_dim", [(12, 10), (64, 33), (300, 20), (520, 6)])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_the_memory_keeps_a_far_write(pkg, compute, key_dim, value_dim):
    """Forget gates near one: what two tokens wrote up to 419 tokens back decides the read-out -- whole, across chunk edges and
    batches of tokens, with the last tokens decoded, and all decoded; without either of them the row is a different one."""
    S, O = pkg.synth, oracle()
    cfg, w, A, B, C, fill = needle_mlstm(S, key_dim, value_dim)
    wd = w64(w)
    n = 420 if key_dim < 100 else 150
    plan = make_plan(pkg, cfg, w, ctx=512, batch=64, compute=compute)
    bound = tol(compute, cfg)
    try:
        toks = [fill[(7 * t + 3) % len(fill)] for t in range(n)]
        toks[n - 1] = A
        toks[30] = C
        without = O.forward(cfg, wd, toks)[n - 1]
        for at in (0, 1, 15, 16, 63, 64, n - 2):
            t2 = list(toks)
            t2[at] = B
            ref = O.forward(cfg, wd, t2)[n - 1]
            assert rel_rms(ref, without) > 0.1, "the planted write has teeth"
            assert rel_rms(prefill_all(plan, t2, 64)[n - 1], ref) <= bound, f"prompt, write at {at}"
            assert rel_rms(portions(plan, t2, [3, 64, 2, n - 90], 64)[n - 1], ref) <= bound, f"portions, write at {at}"
        plan.decode_sequence(t2, n, 0, feedback=False)
        assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref) <= 4 * TOL_DECODE  # hundreds of steps of a state that forgets nothing
    finally:
        plan.free()


def _check_f32(pkg, cfg, w, toks, what, sizes=(1, 2, 3, 2)):
    O = oracle()
    ref_lg, ref_tr = O.forward(cfg, w64(w), toks, return_layers=True)
    plan = make_plan(pkg, cfg, w, batch=64, compute="float32")
    try:
        lg, tr = plan.forward_batch_logits(toks, 0, list(range(len(toks))), want_trace=True)
        assert rel_rms(tr[0][:5], ref_tr[0][:5]) <= tol("float32", cfg), what + ": first tokens"
        for r in range(len(ref_tr)):
            assert rel_rms(tr[r], ref_tr[r]) <= tol("float32", cfg), f"{what}: layer {r}"
        assert_rows(lg, ref_lg, tol("float32", cfg), what)
        assert_rows(portions(plan, toks, list(sizes), 64), ref_lg, tol("float32", cfg), what + " (portions, decode)")
    finally:
        plan.free()
    return ref_lg, ref_tr


def test_embedding_alone(pkg):
    """A layer that adds nothing: the stream is the embedding.  Bigram rows of every residue (one bucket, two, more buckets than
    products, factors of one, factors above the bucket count and above 32 bits), the first token's own row, positions far from zero,
    an even and an odd width; and the logits tell two orders of the same tokens apart."""
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(3)
    toks = rng.integers(0, 60, 62).tolist()
    for E, bigram, scale in [(40, (1, 3, 5), 1.0), (40, (2, 1, 1), 0.3), (41, (9973, 31, 7), 2.0), (24, (17, 2654435761, 40503), 1.0), (30, None, 3.0)]:
        cfg = S.kegasun_config(E, 60, [S.kegasun_mlstm(1, 4, 4, None)], scale=scale, bigram=bigram)
        w = S.kegasun_weights(cfg, 5)
        w["l0.mix.o"][:] = 0.0
        lg, tr = _check_f32(pkg, cfg, w, toks, f"width {E}, bigram {bigram}")
        assert np.allclose(tr[0], O.embedding(cfg, w64(w), toks), atol=1e-12)
    plan = make_plan(pkg, cfg := S.kegasun_config(64, 60, [S.kegasun_mlstm(1, 4, 4, None)]), w := S.kegasun_weights(cfg, 5), ctx=3000, batch=512, compute="float32")
    try:
        long = rng.integers(0, 60, 3000).tolist()
        ref = O.forward(cfg, w64(w), long)
        for c in range(0, 2560, 512):
            plan.forward_batch_prefill(long[c:c + 512], c)
        lg, _ = plan.forward_batch_logits(long[2560:], 2560, [0, 200, 439])
        assert_rows(lg, ref[[2560, 2760, 2999]], 5e-5, "positions in the thousands")
    finally:
        plan.free()


def test_each_attention_mechanism_alone(pkg):
    """Weights that make one mechanism of the latent attention matter (FP32, prefill and decode): sinks above and far below the scores, on one head only; closed,
    open and token-dependent gates per head; latent norms of both signs; a score scale far from key_size^-1/2; a window of one (the output
    is then the token's own value, less the sink's share); windows at and above the sequence length; latents of one entry."""
    S = pkg.synth
    rng = np.random.default_rng(10)
    toks = rng.integers(0, 60, 50).tolist()
    A = S.kegasun_attention
    cases = {"sink_high": A(4, 8, 6, 10, 12, 9), "sink_low": A(4, 8, 6, 10, 12, 9), "sink_one_head": A(4, 8, 6, 10, 12, 9), "gates_closed": A(4, 8, 6, 10, 12, 9), "gates_token": A(4, 8, 6, 10, 12, 9),
             "norm_signs": A(4, 8, 6, 10, 12, 9), "scale": A(2, 8, 6, 10, 12, 20, scale=3.0), "window_one": A(2, 8, 6, 10, 12, 1), "window_length": A(2, 8, 6, 10, 12, 50), "window_long": A(2, 8, 6, 10, 12, 5000),
             "rank_one": A(3, 4, 5, 1, 1, 17), "one_head": A(1, 33, 70, 10, 12, 17), "many_heads": A(17, 2, 1, 9, 5, 6)}
    for case, layer in cases.items():
        cfg = S.kegasun_config(40, 60, [layer])
        w = S.kegasun_weights(cfg, 16)
        if case == "sink_high":
            w["l0.mix.sink"][:] = 6.0
        if case == "sink_low":
            w["l0.mix.sink"][:] = -40.0
        if case == "sink_one_head":
            w["l0.mix.sink"][:] = [-30.0, 9.0, -30.0, 0.0]
        if case == "gates_closed":
            w["l0.mix.g"][:2], w["l0.mix.g"][2:] = 0.0, w["l0.mix.g"][2:] * 30.0
        if case == "gates_token":
            w["l0.mix.g"] *= 5.0
        if case == "norm_signs":
            w["l0.mix.dq.norm"][::2] *= -3.0
            w["l0.mix.dkv.norm"][1::3] *= -0.2
        _check_f32(pkg, cfg, bf16_values(w), toks, case)


def test_each_memory_mechanism_alone(pkg):
    """The same for the matrix memory: forget gates near zero and near one; input gates far below zero (the running maximum starts at zero,
    not at minus infinity: the first tokens write little and the floor of the denominator decides) and far above; queries so small that the
    floor decides everywhere, and so large that it never does; a cap that binds; key sizes 1, 15, 16, 17, 100, 256, 257, 513; value sizes
    1, 16, 17; a norm weight of both signs."""
    S = pkg.synth
    rng = np.random.default_rng(12)
    toks = rng.integers(0, 60, 37).tolist()
    M = S.kegasun_mlstm
    cases = {"forget": M(3, 10, 8), "keep": M(3, 10, 8), "quiet": M(3, 10, 8), "loud": M(3, 10, 8), "small_q": M(2, 10, 8), "large_q": M(2, 10, 8), "cap": M(2, 10, 8, gate_cap=1.5), "gates_token": M(4, 10, 8),
             "norm_signs": M(3, 10, 8)} | {f"key_{d}": M(2, d, 9) for d in (1, 15, 16, 17, 100, 256, 257, 513)} | {f"value_{d}": M(2, 8, d) for d in (1, 16, 17, 50)}
    for case, layer in cases.items():
        cfg = S.kegasun_config(40, 60, [layer], eps=1e-4)
        w = S.kegasun_weights(cfg, 17)
        if case == "forget":
            w["l0.mix.f.b"][:] = -6.0
        if case == "keep":
            w["l0.mix.f.b"][:] = 14.0
        if case == "quiet":
            w["l0.mix.i.b"][:] = -6.0
        if case == "loud":
            w["l0.mix.i.b"][:] = 9.0
        if case == "small_q":
            w["l0.mix.q"] *= 0.02
        if case == "large_q":
            w["l0.mix.q"] *= 50.0
        if case == "cap":
            w["l0.mix.i"] *= 6.0
            w["l0.mix.f"] *= 6.0
        if case == "gates_token":
            w["l0.mix.i"] *= 4.0
            w["l0.mix.f"] *= 4.0
        if case == "norm_signs":
            w["l0.mix.norm"][::2] *= -1.5
        _check_f32(pkg, cfg, bf16_values(w), toks, case)


def test_each_feed_forward_alone(pkg):
    """The same for the feed-forwards: biases that decide the choice against the logits (and enter the weights), all experts, one
    expert, more experts than a warp has lanes, more chosen experts than the row kernel keeps in shared memory; a dense layer alone."""
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(14)
    toks = rng.integers(0, 60, 41).tolist()
    X = S.kegasun_moe
    cases = {"bias": X(6, 2, 12), "all_chosen": X(5, 5, 12), "one_expert": X(1, 1, 9), "top_one": X(4, 1, 12), "many": X(70, 3, 8), "many_chosen": X(80, 70, 4), "sharp": X(6, 3, 16), "dense": S.kegasun_dense(33)}
    for case, mlp in cases.items():
        cfg = S.kegasun_config(40, 60, [S.kegasun_mlstm(1, 4, 4, mlp)])
        w = S.kegasun_weights(cfg, 19)
        w["l0.mix.o"] *= 0.1
        if case == "bias":
            w["l0.mlp.router.b"] = np.array([0.0, 9.0, 0.0, 9.5, 0.0, 0.0], dtype=np.float32)
        if case == "sharp":
            w["l0.mlp.router"] *= 4.0
        w = bf16_values(w)
        if case != "dense":
            assert min_margin(O, cfg, w64(w), toks) > 1e-5, case
        _check_f32(pkg, cfg, w, toks, case)


def test_wide_rows(pkg):
    """A residual row of 2048 entries: the single-row launches of the decode step run with more threads per row than the chunk's."""
    S, O = pkg.synth, oracle()
    cfg = S.kegasun_config(2048, 64, [S.kegasun_mlstm(2, 24, 20, S.kegasun_moe(6, 5, 16)), S.kegasun_attention(2, 8, 8, 20, 24, 6, S.kegasun_dense(24))])
    toks = np.random.default_rng(3).integers(0, 64, 12).tolist()
    w = S.kegasun_weights(cfg, 31)
    assert min_margin(O, cfg, w64(w), toks) > 1e-4
    _check_f32(pkg, cfg, w, toks, "wide", sizes=(3, 1, 2))


def test_long_decoding_through_the_device_loop(pkg):
    """300 single-token steps in one call of the device-resident loop (teacher-forced; the previous token of every step comes from the
    step before): the argmax of every step equals the oracle's wherever the oracle's best two logits are not a near-tie, and the
    last logits agree."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)["mixed"]
    toks = np.random.default_rng(10).integers(0, cfg["vocab"], 300).tolist()
    w = decisive_routing(cfg, S.kegasun_weights(cfg, 16), 16)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, ctx=320, batch=1, compute="bfloat16")
    try:
        ids, ms = plan.decode_sequence(toks, len(toks), 0, feedback=False)
        srt = np.sort(ref, axis=1)
        clear = (srt[:, -1] - srt[:, -2]) > 1e-3 * np.abs(ref).max()
        assert clear.sum() > 250 and np.array_equal(ids[clear], ref.argmax(1)[clear])
        assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref[-1]) <= 2 * TOL_DECODE
        assert ms > 0
    finally:
        plan.free()


def test_greedy_generation_through_the_engine(pkg):
    """engine.generate_tokens_layered (chunked prefill, then the decode step with the device-side argmax) reproduces the oracle's
    greedy continuation; the device loop with feedback gives the same ids; the device sampler at temperature 0 too."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)["mixed"]
    w = decisive_routing(cfg, S.kegasun_weights(cfg, 17), 17)
    wd = w64(w)
    prompt = np.random.default_rng(11).integers(0, cfg["vocab"], 19).tolist()
    seq, want = list(prompt), []
    for _ in range(12):
        lg = O.forward(cfg, wd, seq)[-1]
        top = np.sort(lg)
        assert top[-1] - top[-2] > 1e-4, "near-tie in the oracle: pick another seed"
        want.append(int(lg.argmax()))
        seq.append(want[-1])
    plan = make_plan(pkg, cfg, w, ctx=64, batch=5, compute="float32")
    try:
        got = pkg.engine.generate_tokens_layered(plan, prompt, stop_tokens=[], max_tokens=len(prompt) + 11, context_length=64, batch_size=5)
        assert got == want
        stop = want[4]
        got = pkg.engine.generate_tokens_layered(plan, prompt, stop_tokens=[stop], max_tokens=64, context_length=64, batch_size=5)
        assert got == want[:want.index(stop) + 1]
        for c in range(0, len(prompt) - 1, 5):
            plan.forward_batch_prefill(prompt[c:min(c + 5, len(prompt) - 1)], c)
        ids, _ = plan.decode_sequence([prompt[-1]], 12, len(prompt) - 1, feedback=True)
        assert ids.tolist() == want
        sampler = pkg.sampler.select_sampler(cfg["vocab"], 0.0, 0.9, 1)
        got = pkg.engine.generate_tokens_layered(plan, prompt, stop_tokens=[], max_tokens=len(prompt) + 3, context_length=64, batch_size=5, sampler=sampler)
        assert got == want[:4]
        plan.forward_prefill(prompt[0], 0)  # single-token prefill steps keep the previous token too
        for p in range(1, len(prompt) - 1):
            plan.forward_prefill(prompt[p], p)
        assert plan.forward_decode(prompt[-1], len(prompt) - 1, logits=False)[1] == want[0]
        t = plan.forward_decode_sample(prompt[-1], len(prompt) - 1, 1.3, 0.9, 0.4)
        assert 0 <= t < cfg["vocab"]
    finally:
        plan.free()


@pytest.mark.parametrize("wide", [False, True])
def test_random_layer_lists(pkg, wide):
    """Random layer lists with random sizes and constants: whole, random portions, decode."""
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(2031 + wide)
    for trial in range(6 if wide else 14):
        layers = random_layer_list(S, rng, wide)
        E = int(rng.choice([64, 128, 192, 256])) if wide else int(rng.integers(20, 90))
        cfg = S.kegasun_config(E, int(rng.integers(30, 90)), layers, eps=float(rng.choice([1e-6, 1e-5, 1e-3])), scale=float(rng.uniform(0.4, 2.0)),
                               bigram=None if rng.random() < 0.2 else (int(rng.integers(1, 300)), int(rng.integers(1, 300)), int(rng.integers(1, 300))))
        T, batch = (150, 70) if wide else (45, 9)
        toks = rng.integers(0, cfg["vocab"], T).tolist()
        for compute in ("float32", "bfloat16"):
            w = S.kegasun_weights(cfg, 100 + trial)
            if compute == "bfloat16":
                w = settled_weights(S, O, cfg, trial, toks, 0.5 * tol(compute, cfg))
            elif min_margin(O, cfg, w64(w), toks) < 1e-4:
                continue
            ref = O.forward(cfg, w64(w), toks)
            plan = make_plan(pkg, cfg, w, ctx=T + 19, batch=batch, compute=compute)
            try:
                assert_rows(prefill_all(plan, toks, batch), ref, tol(compute, cfg), f"trial {trial} whole")
                sizes = [int(x) for x in rng.integers(1, batch + 1, 5 if not wide else 3)]
                assert_rows(portions(plan, toks, sizes, batch)[:T], ref, tol(compute, cfg), f"trial {trial} portions {sizes}")
            finally:
                plan.free()


def test_bad_arguments_are_refused(pkg):
    S = pkg.synth
    cfg = configs(S)["mixed"]
    w = S.kegasun_weights(cfg, 19)
    for drop in ("bigram", "l0.mix.dq.norm", "l0.mix.sink", "l0.mix.uq", "l1.mix.i.b", "l1.mix.norm", "l1.mlp.router.b", "l1.mlp.e3.up", "l2.norm2", "final.norm"):
        w2 = {k: v for k, v in w.items() if k != drop}
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, cfg, w2)
    for wrong in ("bigram", "l0.mix.g", "l1.mix.f", "l3.mix.norm"):
        w2 = dict(w)
        w2[wrong] = w2[wrong][:-1]
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, cfg, w2)
    for bad in ([S.kegasun_mlstm(2, 8, 8, None, gate_cap=0.0)], [S.kegasun_attention(2, 8, 8, 6, 6, 0)], [S.kegasun_mlstm(2, 8, 8, S.kegasun_moe(3, 4, 8))]):
        c = S.kegasun_config(64, 96, bad)
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, c, S.kegasun_weights(c, 1))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_steps(pkg, tmp_path, dtype):
    """bin/trace_run on a model directory: steps longer than --chunk, of two tokens and of one, wanted places out of order, steps
    that want nothing, two requests one after the other on one plan (the second starts from an empty state)."""
    import json
    import os
    import subprocess
    import sys

    S, O = pkg.synth, oracle()
    cfg = configs(S)["tiles_a"]
    rng = np.random.default_rng(13)
    reqs = {"a": rng.integers(0, cfg["vocab"], 61).tolist(), "b": rng.integers(0, cfg["vocab"], 9).tolist()}
    w = settled_weights(S, O, cfg, 23, reqs["a"], 0.02)
    assert rounding_shift(O, cfg, w64(w), reqs["b"]) < 0.02
    mdir = str(tmp_path / "model")
    S.write_model_dir(mdir, cfg, w)
    ref = {k: O.forward(cfg, w64(w), v) for k, v in reqs.items()}
    plan_steps = [("a", 37, [36, 0, 5]), ("a", 2, []), ("a", 20, [19, 18]), ("a", 1, [0]), ("a", 1, []), ("b", 1, [0]), ("b", 8, [7, 3])]
    lines, expect, at = [], {}, {"a": 0, "b": 0}
    for n, (rid, count, want) in enumerate(plan_steps):
        lo = at[rid]
        at[rid] = lo + count
        end = [rid] if at[rid] == len(reqs[rid]) else []
        lines.append(json.dumps({"step": n, "entries": [{"id": rid, "tokens": reqs[rid][lo:lo + count], "want": want}], "end": end}))
        if want:
            expect[n] = np.stack([ref[rid][lo + k] for k in want])
    out = str(tmp_path / "out")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", mdir, "--dtype", dtype, "--out", out, "--max-tokens", "64",
                        "--chunk", "16"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == ["done %d" % n for n in range(len(plan_steps))]
    for n in range(len(plan_steps)):
        path = os.path.join(out, "%d.f32" % n)
        if n in expect:
            got = np.fromfile(path, dtype="<f4").reshape(expect[n].shape)
            assert_rows(got, expect[n], tol(dtype, cfg), f"step {n}")
        else:
            assert not os.path.exists(path)
