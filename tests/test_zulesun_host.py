"""CPU tests of the Zulesun support code: config.json registry and the C-ABI structures, synthetic model directories, and
properties of the float64 oracle the GPU tests compare against, one mechanism at a time."""
import ctypes
import math

import numpy as np
import pytest

from zulesun_util import configs, decisive_routing, min_margin, needle_chunk, needle_lightning, needle_scan, oracle, random_layer_list, rel_rms, w64


def test_config_registry_and_abi_structs(pkg, tmp_path):
    S = pkg.synth
    cfg = configs(S)["mixed"]
    w = S.zulesun_weights(cfg, 0)
    d = str(tmp_path / "m")
    S.write_model_dir(d, cfg, w)
    m = pkg.load_model(d, 77)
    c = m.configuration
    assert m.model_type == "ZULESUN" and c.arch == pkg.loader.ARCH_ZULESUN and c.context_length == 77
    assert (c.width, c.vocab_size, c.n_layers, c.block, c.loop, c.norm_eps, c.embedding_scale, c.side_dim) == (64, 96, 4, "sandwich", None, 1e-5, 8.0, 12)
    l0, l1, l2, l3 = c.layers
    assert (l0.mixer, l0.heads, l0.kv_heads, l0.key_dim, l0.value_dim, l0.window, l0.mask_chunked) == ("attention_scan", 4, 2, 16, 12, 7, True)
    assert (l0.score_scale, l0.softcap, l0.qk_norm, l0.gate, l0.gate_per_head, l0.sink, l0.qkv_bias) == (0.25, 25.0, True, True, False, False, False)
    assert (l0.rope_dims, l0.rope_layout, l0.rope_base, l0.rope_factor, l0.branch_scale) == (8, "half", 10000.0, 4.0, (0.9, 1.2))
    assert (l0.scan_inner, l0.scan_state, l0.scan_rank, l0.conv_taps, l0.ff_kind, l0.ff_dim, l0.ff_act) == (40, 6, 5, 4, "dense_plain", 80, "relu2")
    assert (l1.mixer, l1.heads, l1.key_dim, l1.value_dim, len(l1.decay), l1.gate) == ("lightning", 3, 20, 28, 3, True)
    assert (l1.ff_kind, l1.ff_dim, l1.ff_experts, l1.ff_top, l1.ff_act, l1.moe_router, l1.moe_groups, l1.moe_keep, l1.moe_plain) == ("moe", 24, 6, 2, "silu", "softmax_groups", 3, 2, False)
    assert (l2.moe_groups, l2.moe_keep, l3.decay) == (1, 1, (0.5, 0.995))
    assert m.tensors["side.embed"][1] == (48, 96) and m.tensors["l0.mix.left.q.norm"][1] == (64,) and m.tensors["l0.mix.right.A_log"][1] == (6, 40) and "l1.mix.decay" not in m.tensors
    lc, specs = pkg.plan.make_layered_config(m, "float32")
    assert (lc.arch, lc.block, lc.compute, lc.loop_times, lc.side_dim) == (8, 0, 1, -1, 12)
    s0, s1 = specs[0], specs[1]
    assert (s0.mixer, s0.window, s0.mask_chunked, s0.qk_norm, s0.gate, s0.sink, s0.rope_dims, s0.rope_factor, s0.ff_kind, s0.ff_act) == (8, 7, 1, 1, 1, 0, 8, 4.0, 3, 4)
    assert (s0.scan_inner, s0.scan_state, s0.scan_rank, s0.conv_taps) == (40, 6, 5, 4) and list(s0.branch_scale) == pytest.approx([0.9, 1.2])
    assert (s1.mixer, s1.ff_kind, s1.ff_act, s1.moe_router, s1.moe_groups, s1.moe_keep) == (7, 2, 1, 3, 3, 2)
    assert ctypes.sizeof(pkg.native.LayerSpec) == 53 * 4 and ctypes.sizeof(pkg.native.LayeredConfig) == 23 * 4
    # the decays reach the plan as FP32 tensors of their own
    k = pkg.plan.layered_constants(m)
    assert sorted(k) == ["l1.mix.decay", "l3.mix.decay"] and k["l3.mix.decay"][1] == (2,)
    assert np.array_equal(k["l3.mix.decay"][2].view("<f4"), np.asarray([0.5, 0.995], dtype="<f4"))
    # in-memory model = on-disk model
    mm = S.zulesun_model(cfg, w, 77)
    assert mm.configuration == c and all(np.array_equal(mm.tensors[k][2], m.tensors[k][2]) for k in m.tensors)
    # absent optional keys: no mask, no scaling, no rotation, no cap, no groups, no feed-forward, no token input
    bare = S.zulesun_config(32, 40, [S.zulesun_parallel(2, 1, 8, 8, 3, 8, 2, 2, 2, S.zulesun_moe(3, 2, 4)), S.zulesun_lightning(1, 4, 4)], side=None)
    left = bare["layers"][0]["mixer"]["left"]
    del left["mask"], left["rot"], left["softcap"], bare["layers"][0]["mlp"]["router"]["groups"], bare["layers"][1]["mlp"]
    b = pkg.loader.zulesun_configuration(bare, {}, 8)
    b0 = b.layers[0]
    assert (b.side_dim, b0.window, b0.mask_chunked, b0.rope_dims, b0.softcap, b0.moe_groups, b0.moe_keep, b.layers[1].ff_dim) == (0, 8, False, 0, 0.0, 1, 1, 0)
    # unknown mixer / feed-forward kinds and decays that do not fit the heads are refused
    for bad in (dict(cfg["layers"][0], type="delta"), dict(cfg["layers"][0], mlp={"kind": "gated"}), S.zulesun_lightning(2, 4, 4, None, decay=[0.5])):
        with pytest.raises(pkg.loader.UnsupportedModel):
            pkg.loader.zulesun_configuration(dict(cfg, layers=[bad]), {}, 8)
    # the earlier designs keep their defaults
    p = pkg.loader.pibidra_configuration(S.pibidra_config(32, 40, [S.pibidra_layer(2, 1, 8, 8, 4, 16)]), {"l0.mix.rel": (8, 2)}, 8)
    assert (p.layers[0].mask_chunked, p.layers[0].rope_factor, p.layers[0].decay, p.layers[0].branch_scale, p.side_dim) == (False, 0.0, (), (1.0, 1.0), 0)


def test_norms_and_token_input():
    O = oracle()
    rng = np.random.default_rng(1)
    v = rng.standard_normal((4, 9)) * 3.0
    assert np.allclose(O.block_norm(v, np.zeros(9), 0.0), v / np.sqrt((v * v).mean(-1, keepdims=True)))
    assert np.allclose(O.block_norm(v, np.full(9, -1.0), 1e-5), 0.0) and np.allclose(O.rms_norm(v, np.zeros(9), 1e-5), 0.0)   # one is a weight around one, the other around zero
    assert np.all(np.abs(O.block_norm(v * 1e-6, np.zeros(9), 1e-2)) < 1e-3)                                                   # eps sits inside the root
    assert O.gelu_tanh(np.array([0.0, 30.0, -30.0])).tolist() == [0.0, 30.0, 0.0] and O.gelu_tanh(np.array([1.0]))[0] == pytest.approx(0.841192, abs=1e-5)
    w = {"side.embed": rng.standard_normal((6, 9)), "a.side.gate": rng.standard_normal((3, 9)), "a.side.proj": rng.standard_normal((9, 3)), "a.side.norm": np.ones(9)}
    y = O.token_side(v, [2, 5, 2, 0], w, "a.", 1, 3, 0.0)
    g = O.gelu_tanh(v[1] @ w["a.side.gate"].T) * w["side.embed"][5, 3:6]
    assert np.allclose(y[1] * np.sqrt(((w["a.side.proj"] @ g) ** 2).mean()), w["a.side.proj"] @ g) and np.allclose((y * y).mean(-1), 1.0)
    assert not np.allclose(O.token_side(v, [2, 5, 2, 0], w, "a.", 2, 3, 0.0), y)


def test_lightning_pieces():
    O = oracle()
    rng = np.random.default_rng(4)
    T, d, dv = 9, 3, 4
    q, k, v = rng.standard_normal((T, 2, d)), rng.standard_normal((T, 2, d)), rng.standard_normal((T, 2, dv))
    dec = [0.7, 0.99]
    out = O.lightning_scan(q, k, v, dec)
    for a in range(2):
        P = np.tril(q[:, a] @ k[:, a].T) * np.tril(np.float_power(dec[a], np.arange(T)[:, None] - np.arange(T)[None, :]))   # the closed form
        assert np.allclose(out[:, a], P @ v[:, a])
    assert np.allclose(O.lightning_scan(q, k, v, [0.0, 0.0]), np.einsum("thd,thd->th", q, k)[:, :, None] * v)               # nothing but the token itself
    E, H = 10, 2
    w = {n: rng.standard_normal((r, E)) for n, r in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv))} | {"norm": np.ones(H * dv), "o": np.eye(H * dv)}
    h = rng.standard_normal((T, E))
    m = {"heads": H, "dim": d, "vdim": dv, "decay": dec}
    y = O.mixer_lightning(h, w, "", m, 1e-12) / O.sigmoid(h @ w["g"].T)
    assert np.allclose((y ** 2).mean(-1), 1.0, rtol=1e-3) and not np.allclose((y.reshape(T, H, dv) ** 2).mean(-1), 1.0, rtol=1e-2)   # one statistic over all heads
    silent = O.mixer_lightning(h, dict(w, v=np.zeros((H * dv, E))), "", m, 1e-5)
    assert np.allclose(silent, 0.0)                                                                                        # silu(0) = 0


def test_chunked_attention_pieces():
    O = oracle()
    m = O.chunk_mask(7, 3)
    assert m.sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1] and m[5, 3] and not m[5, 2] and not m[3, 4]
    rng = np.random.default_rng(2)
    x = rng.standard_normal((5, 2, 6))
    r = O.rotate_half(x, {"dims": 4, "base": 100.0, "scaling": {"factor": 2.0}})
    assert np.array_equal(r[..., 4:], x[..., 4:]) and np.array_equal(r[0], x[0])
    a = 3 * 100.0 ** (-2.0 / 4) / 2.0
    assert np.allclose(r[3, :, 1], x[3, :, 1] * math.cos(a) - x[3, :, 3] * math.sin(a)) and np.allclose(r[3, :, 3], x[3, :, 3] * math.cos(a) + x[3, :, 1] * math.sin(a))
    assert np.allclose(O.rotate_half(x, {"dims": 4, "base": 100.0})[4, :, 0], x[4, :, 0] * math.cos(4) - x[4, :, 2] * math.sin(4))
    assert np.array_equal(O.rotate_half(x, {"dims": 0, "base": 100.0}), x)
    assert np.abs(O.soft_cap(np.array([1e3, -1e3]), 5.0)).max() <= 5.0 and O.soft_cap(1.5, None) == 1.5
    E, H, G, d, dv, T = 12, 4, 2, 4, 3, 9
    cfg = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "mask": {"size": 1}, "rot": {"dims": 2, "base": 10.0}, "scale": 0.5, "softcap": 4.0}
    w = {"q": rng.standard_normal((H * d, E)), "k": rng.standard_normal((G * d, E)), "v": rng.standard_normal((G * dv, E)), "g": rng.standard_normal((H * dv, E)), "q.norm": rng.standard_normal(H * d),
         "k.norm": rng.standard_normal(G * d), "o": np.eye(H * dv)}
    h = rng.standard_normal((T, E))
    own = np.repeat((h @ w["v"].T).reshape(T, G, dv), H // G, axis=1).reshape(T, -1) * O.sigmoid(h @ w["g"].T)
    assert np.allclose(O.chunked_attention(h, w, "", cfg, 1e-5), own)                       # chunks of one: the token's own gated value
    base = O.chunked_attention(h, w, "", dict(cfg, mask={"size": 4}), 1e-5)
    far = h.copy()
    far[2] += 1.0
    moved = np.abs(O.chunked_attention(far, w, "", dict(cfg, mask={"size": 4}), 1e-5) - base).max(-1) > 1e-9
    assert moved.tolist() == [False, False, True, True] + [False] * 5                        # seen to the end of its chunk
    big = dict(w, q=w["q"] * 7.0, k=w["k"] * 0.2)
    assert np.allclose(O.chunked_attention(h, big, "", dict(cfg, mask={"size": 4}), 0.0), O.chunked_attention(h, w, "", dict(cfg, mask={"size": 4}), 0.0))   # both projections are normed


def test_selective_scan_pieces():
    O = oracle()
    rng = np.random.default_rng(3)
    x = rng.standard_normal((6, 2))
    taps = rng.standard_normal((2, 3))
    c = O.causal_conv(x, taps, np.array([0.5, -1.0]))
    assert np.allclose(c[0], x[0] * taps[:, 2] + [0.5, -1.0]) and np.allclose(c[4], x[2] * taps[:, 0] + x[3] * taps[:, 1] + x[4] * taps[:, 2] + [0.5, -1.0])
    T, I, N = 7, 3, 2
    u, dt, B, C = rng.standard_normal((T, I)), np.abs(rng.standard_normal((T, I))), rng.standard_normal((T, N)), rng.standard_normal((T, N))
    A, D = -np.abs(rng.standard_normal((I, N))), rng.standard_normal(I)
    y = O.selective_scan(u, dt, B, C, A, D)
    t, ch = 5, 1
    want = D[ch] * u[t, ch] + sum(dt[s, ch] * u[s, ch] * sum(math.exp(A[ch, n] * dt[s + 1:t + 1, ch].sum()) * B[s, n] * C[t, n] for n in range(N)) for s in range(t + 1))
    assert y[t, ch] == pytest.approx(want)                                                   # the closed form
    assert np.allclose(O.selective_scan(u, dt * 0.0, B, C, A, D), u * D) and np.allclose(O.softplus(np.array([0.0, 50.0, -50.0])), [math.log(2.0), 50.0, 0.0])
    E = 5
    w = {"in": rng.standard_normal((2 * I, E)), "conv": rng.standard_normal((I, 2)), "conv.b": rng.standard_normal(I), "x": rng.standard_normal((1 + 2 * N, I)), "dt": rng.standard_normal((I, 1)),
         "dt.b": rng.standard_normal(I), "A_log": rng.standard_normal((I, N)), "D": D, "o": np.eye(I)}
    h = rng.standard_normal((T, E))
    m = {"inner": I, "state": N, "dt_rank": 1}
    full = O.mamba(h, w, "", m)
    assert np.allclose(O.mamba(h[:4], w, "", m), full[:4]) and full.shape == (T, I)
    closed = w["in"].copy()
    closed[I:] = 0.0
    assert np.allclose(O.mamba(h, dict(w, **{"in": closed}), "", m), 0.0)                    # silu(z) gates the result


def test_feed_forwards_and_router():
    O = oracle()
    rng = np.random.default_rng(5)
    E, X, F, T = 8, 6, 6, 9
    w = {"router": rng.standard_normal((X, E)), "up": rng.standard_normal((F, E)), "down": rng.standard_normal((E, F))}
    for e in range(X):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = rng.standard_normal((F, E)), rng.standard_normal((F, E)), rng.standard_normal((E, F))
    h = rng.standard_normal((T, E))
    s = np.exp(h @ w["router"].T)
    s /= s.sum(-1, keepdims=True)
    assert np.allclose(O.ff_dense(h, w, ""), (np.maximum(h @ w["up"].T, 0.0) ** 2) @ w["down"].T)
    ids, wts = O.moe_route(h, w, "", {"experts": X, "top": 2, "groups": {"count": 3, "keep": 1}})
    for t in range(T):
        g = int(s[t].argmax()) // 2
        assert sorted(ids[t]) == [2 * g, 2 * g + 1] and np.allclose(wts[t], s[t][ids[t]])     # both experts of the best group, however small the second one's score
    ids, wts = O.moe_route(h, w, "", {"experts": X, "top": 3})
    assert np.array_equal(ids, np.argsort(-s, -1)[:, :3]) and np.all(wts.sum(-1) < 1.0)       # no groups: the three largest, not renormalised
    full = O.ff_moe(h, w, "", {"router": {"experts": X, "top": X, "groups": {"count": 2, "keep": 2}}})
    assert np.allclose(full, sum(s[:, e:e + 1] * O.expert(h, w, f"e{e}.") for e in range(X)))
    m = []
    O.moe_route(h, w, "", {"experts": X, "top": 2, "groups": {"count": 3, "keep": 2}}, m)
    assert len(m) == T and min(m) > 0.0


def test_whole_stack_is_causal_and_chunked(pkg):
    S, O = pkg.synth, oracle()
    for name in ("mixed", "odd"):
        cfg = configs(S)[name]
        w = w64(S.zulesun_weights(cfg, 3))
        toks = np.random.default_rng(6).integers(0, cfg["vocab"], 15).tolist()
        base = O.forward(cfg, w, toks)
        other = list(toks)
        other[9] = (other[9] + 1) % cfg["vocab"]
        moved = np.abs(O.forward(cfg, w, other) - base).max(-1) > 1e-9
        assert not moved[:9].any() and moved[9] and moved[10]
    # attention alone forgets at a chunk's edge: scans weighted with zero, two layers with chunks of 4 and 6 reach to the end of the chunk of the chunk
    cfg = S.zulesun_config(24, 40, [S.zulesun_parallel(2, 1, 8, 8, c, 8, 2, 2, 2, None, branch_scale=(1.0, 0.0)) for c in (4, 6)], side=None)
    w = w64(S.zulesun_weights(cfg, 3))
    toks = np.random.default_rng(7).integers(0, 40, 20).tolist()
    other = [toks[0], (toks[1] + 1) % 40] + toks[2:]
    moved = np.abs(O.forward(cfg, w, other) - O.forward(cfg, w, toks)).max(-1) > 1e-12
    assert moved.tolist() == [False] + [True] * 5 + [False] * 14


def test_planted_models_have_teeth(pkg):
    S, O = pkg.synth, oracle()
    cfg, w, A, B, fill = needle_chunk(S, 20)
    toks = [fill[(7 * t + 3) % len(fill)] for t in range(60)]
    toks[59] = A
    plain = O.forward(cfg, w64(w), toks)[59]
    for at, seen in ((40, True), (39, False), (58, True), (20, False)):
        t2 = list(toks)
        t2[at] = B
        d = rel_rms(O.forward(cfg, w64(w), t2)[59], plain)
        assert d > 0.1 if seen else d < 1e-6
    cfg, w, A, B, C, fill = needle_lightning(S)
    toks = [fill[(7 * t + 3) % len(fill)] for t in range(60)]
    toks[59], toks[30] = A, C
    plain = O.forward(cfg, w64(w), toks)[59]
    for at in (0, 15, 58):
        t2 = list(toks)
        t2[at] = B
        assert rel_rms(O.forward(cfg, w64(w), t2)[59], plain) > 0.1
    for state in (1, 5, 40):
        cfg, w, A, B, fill = needle_scan(S, state)
        toks = [fill[(7 * t + 3) % len(fill)] for t in range(60)]
        toks[59] = A
        plain = O.forward(cfg, w64(w), toks)[59]
        for at in (0, 15, 55):
            t2 = list(toks)
            t2[at] = B
            assert rel_rms(O.forward(cfg, w64(w), t2)[59], plain) > 0.1


def test_decisive_routers_and_random_lists(pkg):
    S, O = pkg.synth, oracle()
    rng = np.random.default_rng(1)
    for name in ("mixed", "tiles_a", "tiles_b"):
        cfg = configs(S)[name]
        w = decisive_routing(cfg, S.zulesun_weights(cfg, 2), 2)
        assert min_margin(O, cfg, w64(w), rng.integers(0, cfg["vocab"], 40).tolist()) > 0.15
    for wide in (False, True):
        for _ in range(5):
            cfg = S.zulesun_config(64, 40, random_layer_list(S, rng, wide))
            c = pkg.loader.zulesun_configuration(cfg, {}, 32)
            assert c.layer_runs() == len(cfg["layers"])
