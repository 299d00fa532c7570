"""CPU tests of the Kegasun support code: config.json registry and the C-ABI structures, synthetic model directories, and
properties of the float64 oracle the GPU tests compare against, one mechanism at a time."""
import ctypes
import math

import numpy as np
import pytest

from kegasun_util import configs, decisive_routing, min_margin, needle_attention, needle_mlstm, oracle, random_layer_list, rel_rms, w64


def test_config_registry_and_abi_structs(pkg, tmp_path):
    S = pkg.synth
    cfg = configs(S)["mixed"]
    w = S.kegasun_weights(cfg, 0)
    d = str(tmp_path / "m")
    S.write_model_dir(d, cfg, w)
    m = pkg.load_model(d, 77)
    c = m.configuration
    assert m.model_type == "KEGASUN" and c.arch == pkg.loader.ARCH_KEGASUN and c.context_length == 77
    assert (c.width, c.vocab_size, c.n_layers, c.block, c.loop, c.norm_eps, c.embedding_scale, c.bigram, c.sinusoid_base) == (64, 96, 4, "layernorm", None, 1e-5, 0.75, (101, 7, 5), 10000.0)
    l0, l1, l2, l3 = c.layers
    assert (l0.mixer, l0.heads, l0.key_dim, l0.value_dim, l0.q_rank, l0.kv_rank, l0.window, l0.rot_dim, l0.kv_from) == ("latent_attention", 4, 16, 12, 24, 20, 7, 0, -1)
    assert (l0.sink, l0.sink_learned, l0.gate, l0.gate_per_head, l0.score_scale, l0.ff_kind, l0.ff_dim, l0.ff_act) == (True, True, True, True, 0.25, "dense", 80, "silu")
    assert (l1.mixer, l1.heads, l1.key_dim, l1.value_dim, l1.gate_cap, l1.score_scale) == ("mlstm", 3, 20, 28, 15.0, pytest.approx(20 ** -0.5))
    assert (l1.ff_kind, l1.ff_dim, l1.ff_experts, l1.ff_top, l1.ff_act, l1.moe_router, l1.moe_plain) == ("moe", 24, 5, 2, "relu2", "softmax_chosen", True)
    assert (l2.window, l3.gate_cap) == (19, 6.0)
    assert m.tensors["bigram"][1] == (64, 102) and m.tensors["l0.mix.uq"][1] == (24, 64) and m.tensors["l1.mix.norm"][1] == (84,) and "l1.mlp.e0.gate" not in m.tensors
    lc, specs = pkg.plan.make_layered_config(m, "float32")
    assert (lc.arch, lc.block, lc.compute, lc.loop_times, lc.bigram_buckets, lc.bigram_mul_prev, lc.bigram_mul_cur, lc.sinusoid, lc.sinusoid_base) == (7, 4, 1, -1, 101, 7, 5, 1, 10000.0)
    assert (specs[0].mixer, specs[0].sink, specs[0].gate, specs[0].q_rank, specs[0].kv_from, specs[0].ff_kind, specs[0].ff_act) == (2, 2, 2, 24, -1, 1, 1)
    assert (specs[1].mixer, specs[1].gate_cap, specs[1].ff_kind, specs[1].ff_act, specs[1].moe_router, specs[1].moe_plain) == (6, 15.0, 2, 4, 2, 1)
    assert ctypes.sizeof(pkg.native.LayerSpec) == 53 * 4 and ctypes.sizeof(pkg.native.LayeredConfig) == 23 * 4
    # in-memory model = on-disk model
    mm = S.kegasun_model(cfg, w, 77)
    assert mm.configuration == c and all(np.array_equal(mm.tensors[k][2], m.tensors[k][2]) for k in m.tensors)
    # factors beyond the bucket count (and beyond 32 bits) name the same rows
    big = S.kegasun_model(dict(cfg, embedding={"scale": 1.0, "bigram": {"buckets": 101, "mul_prev": 101 * 10 ** 10 + 7, "mul_cur": 5 - 101}}), w, 8)
    lc, _ = pkg.plan.make_layered_config(big)
    assert (lc.bigram_mul_prev, lc.bigram_mul_cur) == (7, 5)
    # absent optional keys: no bigram, no window, no feed-forward
    bare = S.kegasun_config(32, 40, [S.kegasun_attention(2, 8, 8, 8, 8, 3)], bigram=None)
    del bare["layers"][0]["mixer"]["mask"], bare["layers"][0]["mlp"]
    b = pkg.loader.kegasun_configuration(bare, {}, 8)
    assert (b.bigram, b.layers[0].window, b.layers[0].ff_dim) == (None, 8, 0)
    # unknown mixer / feed-forward kinds are refused
    with pytest.raises(pkg.loader.UnsupportedModel):
        pkg.loader.kegasun_configuration(dict(cfg, layers=[dict(cfg["layers"][0], type="delta")]), {}, 8)
    with pytest.raises(pkg.loader.UnsupportedModel):
        pkg.loader.kegasun_configuration(dict(cfg, layers=[dict(cfg["layers"][0], mlp={"kind": "gated"})]), {}, 8)
    # the earlier designs keep their defaults
    p = pkg.loader.pibidra_configuration(S.pibidra_config(32, 40, [S.pibidra_layer(2, 1, 8, 8, 4, 16)]), {"l0.mix.rel": (8, 2)}, 8)
    assert (p.layers[0].q_rank, p.layers[0].moe_plain, p.layers[0].gate_cap, p.bigram, p.sinusoid_base) == (0, False, 0.0, None, 0.0)


def test_embedding_and_layer_norm():
    O = oracle()
    bg = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert O.bigram_rows([4, 4, 5, 0], bg) == [10, (12 + 28) % 10, (12 + 35) % 10, 15 % 10]           # the first token has a row of its own
    P = O.sinusoid(5, 7)
    assert np.array_equal(P[0], [0, 1, 0, 1, 0, 1, 0])
    assert P[3, 0] == pytest.approx(math.sin(3.0)) and P[3, 1] == pytest.approx(math.cos(3.0)) and P[3, 4] == pytest.approx(math.sin(3.0 * 10000.0 ** (-4 / 7)))
    rng = np.random.default_rng(1)
    w = {"embed": rng.standard_normal((6, 7)), "bigram": rng.standard_normal((11, 7))}
    x = O.embedding({"width": 7, "embedding": {"scale": 3.0, "bigram": bg}}, w, [2, 5])
    assert np.allclose(x[1], 3.0 * w["embed"][5] + w["bigram"][(6 + 35) % 10] + P[1]) and np.allclose(x[0], 3.0 * w["embed"][2] + w["bigram"][10] + P[0])
    v = rng.standard_normal((4, 9)) * 3.0 + 5.0
    y = O.layer_norm(v, np.ones(9), 0.0)
    assert np.allclose(y.mean(-1), 0.0) and np.allclose((y * y).mean(-1), 1.0)
    assert np.allclose(O.layer_norm(v + 11.0, np.ones(9), 1e-3), O.layer_norm(v, np.ones(9), 1e-3))   # blind to a shift
    assert np.all(np.abs(O.layer_norm(v * 1e-6, np.ones(9), 1e-2)) < 1e-3)                           # eps sits inside the root
    assert np.allclose(O.rms_norm(v, None, 0.0), v / np.sqrt((v * v).mean(-1, keepdims=True)))


def test_window_and_sink():
    O = oracle()
    m = O.window_mask(6, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and m[5, 3] and not m[5, 2] and not m[2, 3]
    rng = np.random.default_rng(2)
    e = rng.standard_normal((6, 6))
    p = O.sink_softmax(e, m, 0.7)
    for i in range(6):
        d = math.exp(0.7) + sum(math.exp(e[i, j]) for j in range(6) if m[i, j])
        assert np.allclose(p[i][m[i]], np.exp(e[i][m[i]]) / d) and not p[i][~m[i]].any()
    assert np.allclose(O.sink_softmax(e, m, -1e3).sum(-1), 1.0) and np.all(O.sink_softmax(e, m, 300.0) < 1e-100)
    assert np.all(np.isfinite(O.sink_softmax(e + 800.0, m, 1.0)))


def test_latent_attention_pieces():
    O = oracle()
    rng = np.random.default_rng(3)
    E, H, d, dv, Rq, R, T = 20, 3, 4, 5, 6, 7, 9
    m = {"heads": H, "dim": d, "vdim": dv, "q_rank": Rq, "kv_rank": R, "mask": {"size": 1}, "scale": 0.5}
    w = {"dq": rng.standard_normal((Rq, E)), "dq.norm": rng.standard_normal(Rq), "uq": rng.standard_normal((H * d, Rq)), "dkv": rng.standard_normal((R, E)), "dkv.norm": rng.standard_normal(R),
         "uk": rng.standard_normal((H * d, R)), "uv": rng.standard_normal((H * dv, R)), "sink": np.full(H, -1e3), "g": rng.standard_normal((H, E)), "o": np.eye(H * dv)}
    h = rng.standard_normal((T, E))
    c = O.rms_norm(h @ w["dkv"].T, w["dkv.norm"], 1e-5)
    own = (c @ w["uv"].T).reshape(T, H, dv) * O.sigmoid(h @ w["g"].T)[:, :, None]
    out = O.mixer_latent_attention(h, w, "", m, 1e-5)
    assert np.allclose(out, own.reshape(T, -1))                                         # window of one, no sink: the token's own gated value
    assert np.allclose(O.mixer_latent_attention(h, dict(w, sink=np.full(H, 1e3)), "", m, 1e-5), 0.0)
    wide = O.mixer_latent_attention(h, w, "", dict(m, mask={"size": 4}), 1e-5)
    far = h.copy()
    far[2] += 1.0
    moved = np.abs(O.mixer_latent_attention(far, w, "", dict(m, mask={"size": 4}), 1e-5) - wide).max(-1) > 1e-9
    assert moved.tolist() == [False, False, True, True, True, True, False, False, False]  # seen up to three tokens later
    scaled = O.mixer_latent_attention(h * 7.0, dict(w, g=w["g"] / 7.0), "", dict(m, mask={"size": 4}), 0.0)
    assert np.allclose(scaled, O.mixer_latent_attention(h, w, "", dict(m, mask={"size": 4}), 0.0))  # both latents are normed


def test_matrix_memory_pieces():
    O = oracle()
    rng = np.random.default_rng(4)
    T, d, dv = 8, 3, 4
    q, k, v = rng.standard_normal((T, 1, d)), rng.standard_normal((T, 1, d)), rng.standard_normal((T, 1, dv))
    i, f = rng.standard_normal((T, 1)), -np.abs(rng.standard_normal((T, 1)))
    out = O.mlstm_scan(q, k, v, i, f)[:, 0]
    # the running maximum cancels: weights exp(i_s + sum of later f) and a denominator of at least one in unscaled units (up to the 1e-6)
    F = np.cumsum(f[:, 0])
    for t in range(T):
        wts = np.array([math.exp(i[s, 0] + F[t] - F[s]) for s in range(t + 1)])
        a = wts * (k[:t + 1, 0] @ q[t, 0])
        assert np.allclose(out[t], (a @ v[:t + 1, 0]) / max(abs(a.sum()), 1.0), rtol=1e-4, atol=1e-6)
    forget = O.mlstm_scan(q, k, v, i, np.full((T, 1), -60.0))[:, 0]
    kq = np.einsum("td,td->t", k[:, 0], q[:, 0]) * np.exp(i[:, 0])
    assert np.allclose(forget, (kq / np.maximum(np.abs(kq), 1.0))[:, None] * v[:, 0], rtol=1e-4, atol=1e-5)   # nothing but the token itself
    quiet = O.mlstm_scan(q, k, v, np.full((T, 1), -30.0), np.zeros((T, 1)))
    assert np.abs(quiet).max() < 1e-10                                                  # the maximum starts at zero: quiet inputs stay small
    ig, fg = O.mlstm_gates(np.ones((1, 2)) * 100.0, {"i": np.array([[1.0, 1.0]]), "i.b": np.zeros(1), "f": np.array([[-1.0, -1.0]]), "f.b": np.zeros(1)}, "", 5.0)
    assert ig[0, 0] == pytest.approx(5.0) and fg[0, 0] == pytest.approx(-math.log1p(math.exp(5.0)))            # both logits are capped
    E, H = 10, 2
    w = {n: rng.standard_normal((r, E)) for n, r in (("q", H * d), ("k", H * d), ("v", H * dv), ("i", H), ("f", H), ("g", H * dv))}
    w |= {"i.b": rng.standard_normal(H), "f.b": rng.standard_normal(H), "norm": np.ones(H * dv), "o": np.eye(H * dv)}
    h = rng.standard_normal((T, E))
    y = O.mixer_mlstm(h, w, "", {"heads": H, "dim": d, "vdim": dv, "gate_cap": 9.0}, 1e-12) / O.sigmoid(h @ w["g"].T)
    assert np.allclose((y.reshape(T, H, dv) ** 2).mean(-1), 1.0, rtol=1e-4)             # every head has unit mean square before the gate


def test_feed_forwards_and_router():
    O = oracle()
    rng = np.random.default_rng(5)
    E, X, F, T = 8, 5, 6, 7
    w = {"router": rng.standard_normal((X, E)), "router.b": np.array([0.0, 0.0, 50.0, 0.0, 0.0])}
    for e in range(X):
        w[f"e{e}.up"], w[f"e{e}.down"] = rng.standard_normal((F, E)), rng.standard_normal((E, F))
    h = rng.standard_normal((T, E))
    z = h @ w["router"].T + w["router.b"]
    ids, wts = O.moe_route(h, w, "", 2)
    assert np.all(ids[:, 0] == 2) and np.allclose(wts.sum(-1), 1.0)
    assert np.allclose(wts[:, 0] / wts[:, 1], np.exp(z[:, 2] - np.take_along_axis(z, ids[:, 1:], -1)[:, 0]))   # softmax over the chosen, bias included
    assert np.allclose(O.moe_route(h, w, "", 1)[1], 1.0)
    assert np.allclose(O.ff_moe(h, w, "", {"router": {"top": 1}}), np.maximum(h @ w["e2.up"].T, 0.0) ** 2 @ w["e2.down"].T)
    full = O.ff_moe(h, w, "", {"router": {"top": X}})
    p = np.exp(z - z.max(-1, keepdims=True))
    p /= p.sum(-1, keepdims=True)
    assert np.allclose(full, sum(p[:, e:e + 1] * O.expert(h, w, f"e{e}.") for e in range(X)))
    assert np.allclose(O.relu_squared(np.array([-2.0, 0.0, 3.0])), [0.0, 0.0, 9.0]) and np.allclose(O.silu(np.array([0.0, 20.0])), [0.0, 20.0])


def test_whole_stack_is_causal_and_windowed(pkg):
    S, O = pkg.synth, oracle()
    for name in ("mixed", "odd"):
        cfg = configs(S)[name]
        w = w64(S.kegasun_weights(cfg, 3))
        toks = np.random.default_rng(6).integers(0, cfg["vocab"], 15).tolist()
        base = O.forward(cfg, w, toks)
        other = list(toks)
        other[9] = (other[9] + 1) % cfg["vocab"]
        moved = np.abs(O.forward(cfg, w, other) - base).max(-1) > 1e-9
        assert not moved[:9].any() and moved[9] and moved[10]
    # attention alone forgets: three layers of windows 1, 12, 33 reach back 0 + 11 + 32 tokens (no bigram in this model)
    cfg = configs(S)["attention_only"]
    w = w64(S.kegasun_weights(cfg, 3))
    toks = np.random.default_rng(7).integers(0, cfg["vocab"], 50).tolist()
    other = [(toks[0] + 1) % cfg["vocab"]] + toks[1:]
    moved = np.abs(O.forward(cfg, w, other) - O.forward(cfg, w, toks)).max(-1) > 1e-12
    assert moved[:44].all() and not moved[44:].any()


def test_planted_models_have_teeth(pkg):
    S, O = pkg.synth, oracle()
    cfg, w, A, B, fill = needle_attention(S, 20)
    toks = [fill[(7 * t + 3) % len(fill)] for t in range(60)]
    toks[59] = A
    plain = O.forward(cfg, w64(w), toks)[59]
    for at, seen in ((59 - 19, True), (59 - 20, False), (58, True)):
        t2 = list(toks)
        t2[at] = B
        d = rel_rms(O.forward(cfg, w64(w), t2)[59], plain)
        assert d > 0.1 if seen else d < 1e-6
    cfg, w, A, B, C, fill = needle_mlstm(S)
    toks = [fill[(7 * t + 3) % len(fill)] for t in range(60)]
    toks[59], toks[30] = A, C
    plain = O.forward(cfg, w64(w), toks)[59]
    for at in (0, 15, 58):
        t2 = list(toks)
        t2[at] = B
        assert rel_rms(O.forward(cfg, w64(w), t2)[59], plain) > 0.1


def test_decisive_routers_and_random_lists(pkg):
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(1)
    for name in ("mixed", "tiles_a", "tiles_b"):
        cfg = configs(S)[name]
        w = decisive_routing(cfg, S.kegasun_weights(cfg, 2), 2)
        assert min_margin(O, cfg, w64(w), rng.integers(0, cfg["vocab"], 40).tolist()) > 0.15
    for wide in (False, True):
        for _ in range(5):
            cfg = S.kegasun_config(64, 40, random_layer_list(S, rng, wide))
            c = pkg.loader.kegasun_configuration(cfg, {}, 32)
            assert c.layer_runs() == len(cfg["layers"])
