"""GPU tests of the Zulesun mechanisms of sandwich-normed layered plans (csrc/sandwich_plan.cuh, csrc/lightning.cuh, csrc/selective.cuh and the
kernels they share with the other layered designs) on small random models, against the float64 oracle (oracle/zulesun_oracle.py, which
shares no code with the product).

Tolerances.  FP32 compute mode and the decode step (FP32 activations in either mode): relative RMS error of a logits row
<= 5e-5 (only the summation order differs): this is the sharp comparison, and every case runs in it.  BF16 compute mode, batched
prefill: GEMM operands are rounded to BF16 and the untrained random layers pass the rounding of every layer on to the next, so the
bound grows with depth: 1.5 % per layer (+ 1 for the classifier).  In BF16 mode the routers never face a close call (see
zulesun_util.decisive_routing), and no read-out of the linear attention is one that rounding may turn (zulesun_util.rounding_shift).  Where a
test plants a key or a write that decides the output, the model has one layer (bound 3 %) and a slip of the cache or the state moves the
row by more than 10 %."""
import numpy as np
import pytest

from zulesun_util import bf16_values, configs, decisive_routing, min_margin, needle_chunk, needle_lightning, needle_scan, oracle, random_layer_list, rel_rms, rounding_shift, settled_weights, w64

pytestmark = pytest.mark.gpu

TOL_DECODE = 5e-5
SETTLED_F32 = 4e-4  # how far disturbances of 2^-17 may move a row that FP32 results are compared with
ALL = ["mixed", "odd", "parallel_only", "lightning_only", "tiles_a", "tiles_b"]


def tol(compute, cfg):
    return 5e-5 if compute == "float32" else 1.5e-2 * (len(cfg["layers"]) + 1)


def weights_for(S, O, cfg, seed, compute, toks):
    """Random weights; in BF16 mode with decisive routers and no read-out that rounding may turn.  In FP32 mode no near-tie of two experts or groups, and no row that tiny disturbances turn."""
    if compute == "bfloat16":
        return settled_weights(S, O, cfg, seed, toks, 0.5 * tol(compute, cfg))
    for k in range(seed, seed + 30):
        w = S.zulesun_weights(cfg, k)
        if min_margin(O, cfg, w64(w), toks) > 1e-4 and rounding_shift(O, cfg, w64(w), toks, 17) < SETTLED_F32:
            return w
    raise AssertionError("near-ties of experts or unsettled rows in the oracle for every seed")


def make_plan(pkg, cfg, weights, ctx=256, batch=16, compute="float32"):
    model = pkg.synth.zulesun_model(cfg, weights, ctx)
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
    """Residual stream after every layer and the logits: each mixer alone (parallel_only, lightning_only) and in every order, with and
    without feed-forwards and token input."""
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
@pytest.mark.parametrize("name", ["mixed", "odd", "parallel_only", "lightning_only"])
def test_portions_of_every_size(pkg, name, compute):
    """The same prompt cut into portions of 1 .. 13 tokens (cuts inside the attention's chunks, inside the convolutions' taps and inside the
    recurrences' batches of tokens), then decoded one by one; the launch capacity (7) is below the portion sizes, so portions are
    cut again, and the rings have just chunk - 1 + 7 slots."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 70).tolist()
    w = weights_for(S, O, cfg, 13, compute, toks)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, ctx=70, batch=7, compute=compute)  # the last token fills the context
    try:
        chunks = [lc["mixer"]["left"]["mask"]["size"] for lc in cfg["layers"] if lc["type"] == "parallel"]
        assert plan.layered_info()[1] == min(70, max([min(x, 70) for x in chunks] + [1]) - 1 + 7)
        for sizes in ([2, 3, 2, 13, 5, 2, 11, 2, 7], [9, 2, 1, 2, 2, 12, 1, 1, 3], [50], [2] * 20, [1, 2, 1, 60]):
            assert_rows(portions(plan, toks, sizes, 7), ref, tol(compute, cfg), f"portions {sizes}")
    finally:
        plan.free()


@pytest.mark.parametrize("name", ["tiles_a", "tiles_b"])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_tensor_core_prefill_shapes(pkg, name, compute):
    """Shapes that take the tcgen05 GEMMs, the tensor-core attention and the chunk-parallel linear attention in BF16 mode: a prompt longer than
    several key tiles and than the rings, whole, in ragged portions, then decoded; then a second request over the same rings."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)[name]
    toks = np.random.default_rng(12).integers(0, cfg["vocab"], 330).tolist()
    w = weights_for(S, O, cfg, 21, compute, toks)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, ctx=340, batch=150, compute=compute)
    try:
        assert_rows(prefill_all(plan, toks, 150), ref, tol(compute, cfg), "whole")
        assert_rows(portions(plan, toks, (65, 2, 129, 1, 5, 3, 64, 2, 20), 150), ref, tol(compute, cfg), "portions")
        assert_rows(prefill_all(plan, toks[:30], 150), ref[:30], tol(compute, cfg), "second request")
    finally:
        plan.free()


def test_state_and_slots_are_reused_across_requests(pkg):
    """Request after request on one plan without clearing anything: a request starts from empty states and convolutions and sees none of
    the earlier keys; kv_reset in between changes nothing."""
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
            for layer in (0, 1):
                assert np.abs(plan.read_buffer("delta_state", 32, layer=layer)).max() > 0
            assert np.abs(plan.read_buffer("conv_state", 40, layer=0)).max() > 0
            if k == 2:
                plan.kv_reset()
                for layer in (0, 1):
                    assert np.abs(plan.read_buffer("delta_state", 32, layer=layer)).max() == 0
                assert np.abs(plan.read_buffer("conv_state", 40, layer=0)).max() == 0
        with pytest.raises(pkg.native.B200Error):
            plan.read_buffer("conv_state", 4, layer=1)
    finally:
        plan.free()


@pytest.mark.parametrize("shape", [(8, 12), (64, 64), (64, 32)])
@pytest.mark.parametrize("chunk", [1, 2, 37, 64, 65, 150])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_chunk_edges_with_a_planted_key(pkg, compute, chunk, shape):
    """One key decides the output.  It sits on the first token of the query's chunk, on the last token of the chunk before, just before
    the query, and a whole chunk back; the queries sit on a chunk's first, second and last token, on both sides of a launch's edge and of the
    ring's last slot -- in a prompt (whole and in portions), with the query decoded after a prefill, and with everything decoded.
    (64, 64) and (64, 32): the tensor-core attention in BF16 mode."""
    S, O = pkg.synth, oracle()
    cfg, w, A, B, fill = needle_chunk(S, chunk, *shape)
    wd = w64(w)
    ctx, batch = 330, 64
    plan = make_plan(pkg, cfg, w, ctx=ctx, batch=batch, compute=compute)
    bound = tol(compute, cfg)
    try:
        ring = plan.layered_info()[1]
        queries = {chunk, 2 * chunk - 1, 2 * chunk, 63, 64, 65, 129, ring, ring + 1, ctx - 1}
        places = {(i, at) for i in queries for at in (i // chunk * chunk, i // chunk * chunk - 1, i - 1, i - chunk, i // chunk * chunk + chunk // 2)} | {(1, 0), (3, 0)}
        for i, at in sorted(places):
            if not 0 <= at < i < ctx:
                continue
            toks = [fill[(7 * t + 3) % len(fill)] for t in range(i + 1)]
            toks[i] = A
            without = O.forward(cfg, wd, toks)[i]
            toks[at] = B
            ref = O.forward(cfg, wd, toks)[i]
            if i // chunk == at // chunk:
                assert rel_rms(without, ref) > 0.1, "the planted key has teeth"
            else:
                assert rel_rms(without, ref) < 1e-9, "a key of another chunk is not seen"
            assert rel_rms(prefill_all(plan, toks, batch)[i], ref) <= bound, f"prompt, query {i}, key at {at}"
            assert rel_rms(portions(plan, toks, [2] * ((i + 1) // 2) if i < 70 else [61, 2, 3, i - 66], batch)[i], ref) <= bound, f"portions, query {i}, key at {at}"
            prefill_all(plan, toks[:i], batch)
            assert rel_rms(plan.forward_decode(toks[i], i)[0], ref) <= bound, f"decoded query {i}, key at {at}"  # the keys came from the prefill kernels
            plan.decode_sequence(toks, i + 1, 0, feedback=False)
            assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref) <= TOL_DECODE, f"all decoded, query {i}, key at {at}"
    finally:
        plan.free()


@pytest.mark.parametrize("key_dim,value_dim", [(12, 10), (64, 64), (128, 33), (300, 20)])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_linear_attention_keeps_a_far_write(pkg, compute, key_dim, value_dim):
    """Decays near one: what two tokens wrote up to 419 tokens back decides the read-out -- whole, across launch edges and
    batches of tokens, with the last tokens decoded, and all decoded; without either of them the row is a different one."""
    S, O = pkg.synth, oracle()
    cfg, w, A, B, C, fill = needle_lightning(S, key_dim, value_dim)
    wd = w64(w)
    n = 420 if key_dim < 200 else 150
    plan = make_plan(pkg, cfg, w, ctx=512, batch=160, compute=compute)
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
            assert rel_rms(prefill_all(plan, t2, 160)[n - 1], ref) <= bound, f"prompt, write at {at}"
            assert rel_rms(portions(plan, t2, [3, 64, 2, n - 90], 160)[n - 1], ref) <= bound, f"portions, write at {at}"
        plan.decode_sequence(t2, n, 0, feedback=False)
        assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref) <= 4 * TOL_DECODE  # hundreds of steps of a state that forgets little
    finally:
        plan.free()


@pytest.mark.parametrize("state,taps", [(1, 1), (5, 3), (16, 4), (40, 2), (130, 5)])
@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_selective_scan_keeps_a_far_write(pkg, compute, state, taps):
    """The same for the selective scan: states that barely decay, one token's write decides what is read up to 419 tokens later."""
    S, O = pkg.synth, oracle()
    cfg, w, A, B, fill = needle_scan(S, state, taps)
    wd = w64(w)
    n = 420 if state < 100 else 150
    plan = make_plan(pkg, cfg, w, ctx=512, batch=64, compute=compute)
    bound = tol(compute, cfg)
    try:
        toks = [fill[(7 * t + 3) % len(fill)] for t in range(n)]
        toks[n - 1] = A
        without = O.forward(cfg, wd, toks)[n - 1]
        for at in (0, 1, 15, 16, 63, 64, n - 2):
            t2 = list(toks)
            t2[at] = B
            ref = O.forward(cfg, wd, t2)[n - 1]
            assert rel_rms(ref, without) > 0.1, "the planted write has teeth"
            assert rel_rms(prefill_all(plan, t2, 64)[n - 1], ref) <= bound, f"prompt, write at {at}"
            assert rel_rms(portions(plan, t2, [3, 64, 2, n - 90], 64)[n - 1], ref) <= bound, f"portions, write at {at}"
        plan.decode_sequence(t2, n, 0, feedback=False)
        assert rel_rms(plan.read_buffer("logits", cfg["vocab"]), ref) <= 4 * TOL_DECODE
    finally:
        plan.free()


@pytest.mark.parametrize("key_dim,value_dim", [(32, 72), (64, 64), (128, 200)])
def test_chunk_parallel_state_is_exact_behind_its_operands(pkg, key_dim, value_dim):
    """The tensor-core form of the linear attention rounds q, k, v to BF16 and nothing else: the state it leaves after 200 tokens in launches of 150 and
    50 (whole and ragged tiles of tokens) is the one that the recurrence over the rounded keys and values gives, to 32-bit accuracy, for
    decays of zero, one, and between."""
    S, O = pkg.synth, oracle()
    decay = [0.0, 0.5, 0.97, 0.9999, 1.0]
    cfg = S.zulesun_config(128, 60, [S.zulesun_lightning(5, key_dim, value_dim, None, decay=decay)], side=None)
    w = S.zulesun_weights(cfg, 41)
    wd = w64(w)
    toks = np.random.default_rng(9).integers(0, 60, 200).tolist()
    h = bf16_values({"h": O.block_norm(wd["embed"][toks] * cfg["embedding"]["scale"], wd["l0.norm1"], 1e-5)})["h"].astype(np.float64)
    k, v = (bf16_values({"x": O.silu(h @ wd[f"l0.mix.{n}"].T)})["x"].astype(np.float64).reshape(200, 5, -1) for n in "kv")
    plan = make_plan(pkg, cfg, w, ctx=256, batch=150, compute="bfloat16")
    try:
        prefill_all(plan, toks, 150)
        got = plan.read_buffer("delta_state", 5 * value_dim * key_dim, layer=0).reshape(5, value_dim, key_dim)
    finally:
        plan.free()
    for a, c in enumerate(decay):
        ref = np.zeros((value_dim, key_dim))
        for t in range(200):
            ref = float(np.float32(c)) * ref + np.outer(v[t, a], k[t, a])
        assert rel_rms(got[a].reshape(-1), ref.reshape(-1)) < 2e-4, f"decay {c}"  # a key or value may round the other way: one in thousands by 2^-9


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


def test_each_attention_mechanism_alone(pkg):
    """Weights that make one mechanism of the attention matter (FP32, prefill and decode; the scan's part weighted with zero): no rotation, a
    full one, of two entries; no scaling, scaling far above and below one; a cap that binds, none; norm weights of both signs and of zero; open,
    closed and token-dependent gates; a score scale far from key_size^-1/2; chunks of one token and above the sequence; one head,
    many heads, every grouping; a branch scale below zero."""
    S = pkg.synth
    rng = np.random.default_rng(10)
    toks = rng.integers(0, 60, 50).tolist()

    def P(H, G, dk, dv, chunk, **kw):
        return S.zulesun_parallel(H, G, dk, dv, chunk, 4, 2, 1, 2, None, **({"branch_scale": (1.0, 0.0)} | kw))

    cases = {"rot_none": P(4, 2, 8, 6, 9, rot_dims=0), "rot_full": P(4, 2, 8, 6, 20, rot_dims=8, factor=None), "rot_two": P(4, 2, 8, 6, 20, rot_dims=2, base=3.0), "factor_large": P(4, 2, 8, 6, 20, factor=50.0),
             "factor_small": P(4, 2, 8, 6, 20, factor=0.3), "cap_binds": P(4, 2, 8, 6, 20, scale=3.0, softcap=1.5), "cap_none": P(4, 2, 8, 6, 20, softcap=0.0), "norm_signs": P(4, 2, 8, 6, 20),
             "norm_zero": P(4, 2, 8, 6, 20), "gates_closed": P(4, 2, 8, 6, 9), "gates_token": P(4, 2, 8, 6, 9), "scale": P(2, 1, 8, 6, 20, scale=3.0), "chunk_one": P(2, 1, 8, 6, 1), "chunk_length": P(2, 1, 8, 6, 50),
             "chunk_long": P(2, 1, 8, 6, 5000), "one_head": P(1, 1, 33, 70, 17), "many_heads": P(18, 3, 2, 1, 6, rot_dims=2), "own_keys": P(5, 5, 4, 3, 11), "negative": P(3, 1, 8, 6, 12, branch_scale=(-1.5, 0.0)),
             "both_branches": P(3, 1, 8, 6, 12, branch_scale=(0.25, 2.0))}
    for case, layer in cases.items():
        cfg = S.zulesun_config(40, 60, [layer], side=None)
        w = S.zulesun_weights(cfg, 16)
        q = "l0.mix.left."
        if case == "norm_signs":
            w[q + "q.norm"][::2] *= -3.0
            w[q + "k.norm"][1::3] *= -0.2
        if case == "norm_zero":
            w[q + "q.norm"][:8] = 0.0
        if case == "gates_closed":
            w[q + "g"][:12], w[q + "g"][12:] = 0.0, w[q + "g"][12:] * 30.0
        if case == "gates_token":
            w[q + "g"] *= 5.0
        if case == "cap_none":
            del layer["mixer"]["left"]["softcap"]
        _check_f32(pkg, cfg, bf16_values(w), toks, case)
    plain = S.zulesun_config(40, 60, [P(4, 2, 8, 6, 20)], side=None)  # no mask at all: every earlier position
    del plain["layers"][0]["mixer"]["left"]["mask"]
    w = S.zulesun_weights(plain, 16)
    ref = S.zulesun_config(40, 60, [P(4, 2, 8, 6, 5000)], side=None)
    got = {}
    for k, cfg in (("plain", plain), ("one chunk", ref)):
        plan = make_plan(pkg, cfg, w, batch=64)
        got[k] = prefill_all(plan, toks, 64)
        plan.free()
    assert np.abs(got["plain"] - got["one chunk"]).max() < 1e-5 * np.abs(got["plain"]).max()


def test_each_scan_mechanism_alone(pkg):
    """The same for the selective scan (the attention's part weighted with zero): one tap and more taps than the first portions have tokens;
    step ranks, state and channel counts on every side of the kernel's lane and register rows; large and vanishing steps; decays near
    zero and near one; no skip term; a convolution bias alone."""
    S = pkg.synth
    rng = np.random.default_rng(12)
    toks = rng.integers(0, 60, 37).tolist()

    def P(inner, state, rank, taps, **kw):
        return S.zulesun_parallel(2, 1, 4, 4, 9, inner, state, rank, taps, None, **({"branch_scale": (0.0, 1.0)} | kw))

    cases = {f"state_{n}": P(20, n, 3, 3) for n in (1, 3, 4, 5, 8, 9, 16, 17, 32, 33, 64, 65, 128, 129, 400)} | {f"inner_{n}": P(n, 6, 3, 3) for n in (1, 7, 64, 65, 130)} | \
            {f"rank_{n}": P(20, 6, n, 3) for n in (1, 8, 40)} | {f"taps_{n}": P(20, 6, 3, n) for n in (1, 2, 9)} | \
            {k: P(24, 8, 4, 3) for k in ("steps_large", "steps_tiny", "decay_fast", "decay_slow", "no_skip", "conv_bias", "gates_token")} | {"scaled": P(24, 8, 4, 3, branch_scale=(0.0, -3.0))}
    for case, layer in cases.items():
        cfg = S.zulesun_config(40, 60, [layer], side=None, eps=1e-4)
        w = S.zulesun_weights(cfg, 17)
        r = "l0.mix.right."
        if case == "steps_large":
            w[r + "dt.b"][:] = 6.0
        if case == "steps_tiny":
            w[r + "dt.b"][:] = -9.0
            w[r + "D"][:] = 0.0
        if case == "decay_fast":
            w[r + "A_log"][:] = 5.0
        if case == "decay_slow":
            w[r + "A_log"][:] = -7.0
        if case == "no_skip":
            w[r + "D"][:] = 0.0
        if case == "conv_bias":
            w[r + "conv"][:] = 0.0
        if case == "gates_token":
            w[r + "in"][24:] *= 4.0
        _check_f32(pkg, cfg, bf16_values(w), toks, case)


def test_each_linear_attention_mechanism_alone(pkg):
    """The same for the decayed linear attention: decays of zero, one half, one, and unequal ones; key sizes on every side of the kernel's
    lane rows; value sizes 1, 16, 17, 50; a norm weight of both signs; a read-out so small that eps decides; token-dependent gates."""
    S = pkg.synth
    rng = np.random.default_rng(13)
    toks = rng.integers(0, 60, 37).tolist()
    L = S.zulesun_lightning
    cases = {"decay_zero": L(3, 10, 8, None, decay=[0.0, 0.0, 0.0]), "decay_one": L(2, 10, 8, None, decay=[1.0, 1.0]), "decay_mixed": L(4, 10, 8, None, decay=[0.0, 0.5, 0.999, 1.0]), "norm_signs": L(3, 10, 8),
             "quiet": L(3, 10, 8), "gates_token": L(3, 10, 8)} | {f"key_{d}": L(2, d, 9) for d in (1, 15, 16, 17, 33, 100, 256, 257, 512)} | {f"value_{d}": L(2, 8, d) for d in (1, 16, 17, 50)}
    for case, layer in cases.items():
        cfg = S.zulesun_config(40, 60, [layer], side=None, eps=1e-4)
        w = S.zulesun_weights(cfg, 18)
        if case == "norm_signs":
            w["l0.mix.norm"][::2] *= -1.5
        if case == "quiet":
            w["l0.mix.v"] *= 0.01
        if case == "gates_token":
            w["l0.mix.g"] *= 5.0
        _check_f32(pkg, cfg, bf16_values(w), toks, case)


def test_each_feed_forward_alone(pkg):
    """The same for the feed-forwards: one group, as many groups as experts, one kept, all kept; a second expert of the best group that a better
    one of a dropped group would beat; all experts, one expert, more experts than a warp has lanes, more chosen experts than the row
    kernel keeps in shared memory; the squared ReLU alone."""
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(14)
    toks = rng.integers(0, 60, 41).tolist()
    X = S.zulesun_moe
    cases = {"one_group": X(6, 2, 12), "groups": X(6, 2, 12, 3, 1), "groups_two": X(12, 3, 8, 4, 2), "group_each": X(5, 2, 12, 5, 3), "all_kept": X(6, 2, 12, 2, 2), "all_chosen": X(5, 5, 12), "one_expert": X(1, 1, 9),
             "many": X(72, 3, 8, 9, 2), "many_groups": X(80, 4, 4, 40, 7), "many_chosen": X(80, 70, 4), "sharp": X(6, 3, 16, 2, 1), "dense": S.zulesun_dense(33), "dense_wide": S.zulesun_dense(300)}
    for case, mlp in cases.items():
        cfg = S.zulesun_config(40, 60, [S.zulesun_lightning(1, 4, 4, mlp)], side=None)
        for seed in range(19, 29):
            w = S.zulesun_weights(cfg, seed)
            w["l0.norm1b"][:] = -0.9
            if case == "sharp":
                w["l0.mlp.router"] *= 4.0
            w = bf16_values(w)
            if min_margin(O, cfg, w64(w), toks) > 1e-5:
                break
        assert min_margin(O, cfg, w64(w), toks) > 1e-5, case
        _check_f32(pkg, cfg, w, toks, case)


def test_token_input_alone(pkg):
    """Layers that add nothing but the token input: sizes of one entry, of no multiple of 4, of whole blocks and above the width; every layer reads its
    own part of the table; norm weights of both signs; behind a layer without a feed-forward."""
    S = pkg.synth
    rng = np.random.default_rng(15)
    toks = rng.integers(0, 60, 33).tolist()
    for D in (1, 7, 64, 100):
        cfg = S.zulesun_config(40, 60, [S.zulesun_lightning(1, 4, 4, None), S.zulesun_lightning(1, 4, 4, S.zulesun_dense(8)), S.zulesun_lightning(1, 4, 4, None)], side=D)
        w = S.zulesun_weights(cfg, 5)
        for i in range(3):
            w[f"l{i}.norm1b"][:] = -1.0
            w[f"l{i}.side.norm"][::3] *= -1.0
        w["l1.norm2b"][:] = -1.0
        ref, tr = _check_f32(pkg, cfg, bf16_values(w), toks, f"token input of {D}")
        assert all(np.abs(tr[i + 1] - tr[i]).max() > 0.05 for i in range(2))


@pytest.mark.parametrize("compute", ["float32", "bfloat16"])
def test_wide_rows(pkg, compute):
    """A residual row of 2048 entries: the single-row launches of the decode step run with more threads per row than the chunk's."""
    S, O = pkg.synth, oracle()
    cfg = S.zulesun_config(2048, 64, [S.zulesun_lightning(2, 24, 20, S.zulesun_moe(6, 5, 16, 2, 2)), S.zulesun_parallel(2, 1, 8, 8, 6, 72, 12, 20, 4, S.zulesun_dense(24))], side=64)
    toks = np.random.default_rng(3).integers(0, 64, 12).tolist()
    w = weights_for(S, O, cfg, 31, compute, toks)
    ref = O.forward(cfg, w64(w), toks)
    plan = make_plan(pkg, cfg, w, batch=16, compute=compute)
    try:
        assert_rows(prefill_all(plan, toks, 16), ref, tol(compute, cfg), "wide")
        assert_rows(portions(plan, toks, (3, 1, 2), 16), ref, tol(compute, cfg), "wide, portions")
    finally:
        plan.free()


def test_long_decoding_through_the_device_loop(pkg):
    """300 single-token steps in one call of the device-resident loop (teacher-forced): the argmax of every step equals the oracle's
    wherever the oracle's best two logits are not a near-tie, and the last logits agree."""
    S, O = pkg.synth, oracle()
    cfg = configs(S)["mixed"]
    toks = np.random.default_rng(10).integers(0, cfg["vocab"], 300).tolist()
    w = decisive_routing(cfg, S.zulesun_weights(cfg, 16), 16)
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
    w = decisive_routing(cfg, S.zulesun_weights(cfg, 17), 17)
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
        for p in range(len(prompt) - 1):  # single-token prefill steps
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
    rng = np.random.default_rng(2041 + wide)
    for trial in range(6 if wide else 14):
        layers = random_layer_list(S, rng, wide)
        E = int(rng.choice([64, 128, 192, 256])) if wide else int(rng.integers(20, 90))
        cfg = S.zulesun_config(E, int(rng.integers(30, 90)), layers, eps=float(rng.choice([1e-6, 1e-5, 1e-3])), scale=float(rng.uniform(0.4, 20.0)),
                               side=None if rng.random() < 0.2 else int(rng.choice([64, 128])) if wide else int(rng.integers(1, 30)))
        T, batch = (150, 70) if wide else (45, 9)
        toks = rng.integers(0, cfg["vocab"], T).tolist()
        for compute in ("float32", "bfloat16"):
            if compute == "bfloat16":
                w = settled_weights(S, O, cfg, trial, toks, 0.5 * tol(compute, cfg))
            else:
                w = S.zulesun_weights(cfg, 100 + trial)
                if min_margin(O, cfg, w64(w), toks) < 1e-4 or rounding_shift(O, cfg, w64(w), toks, 17) > SETTLED_F32:
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
    w = S.zulesun_weights(cfg, 19)
    for drop in ("side.embed", "l0.norm1b", "l0.mix.left.q.norm", "l0.mix.left.g", "l0.mix.right.in", "l0.mix.right.conv.b", "l0.mix.right.A_log", "l0.mix.right.o", "l0.mlp.up", "l1.mix.norm", "l1.mlp.e3.up", "l1.mlp.router",
                 "l2.norm2b", "l3.side.proj", "final.norm"):
        w2 = {k: v for k, v in w.items() if k != drop}
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, cfg, w2)
    for wrong in ("side.embed", "l0.mix.left.o", "l0.mix.right.x", "l0.mix.right.dt", "l0.mix.right.D", "l1.mix.g", "l3.side.gate"):
        w2 = dict(w)
        w2[wrong] = w2[wrong][:-1]
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, cfg, w2)
    P, L, X = S.zulesun_parallel, S.zulesun_lightning, S.zulesun_moe
    for bad in (P(2, 1, 8, 8, 0, 8, 2, 2, 2), P(3, 2, 8, 8, 4, 8, 2, 2, 2), P(2, 1, 8, 8, 4, 8, 600, 2, 2), P(2, 1, 8, 8, 4, 8, 2, 2, 0), P(2, 1, 8, 8, 4, 8, 2, 2, 2, rot_dims=10), L(1, 520, 4), L(2, 8, 8, X(3, 4, 8)), L(2, 8, 8, X(6, 3, 8, 3, 1)),
                L(2, 8, 8, X(6, 2, 8, 4, 1))):
        c = S.zulesun_config(64, 96, [bad])
        with pytest.raises(pkg.native.B200Error):
            make_plan(pkg, c, S.zulesun_weights(c, 1))


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
    w = settled_weights(S, O, cfg, 23, reqs["a"] + reqs["b"], 0.03)
    assert rounding_shift(O, cfg, w64(w), reqs["b"]) < 0.03
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
