"""Shared helpers of the Kegasun tests: small configurations, weights with planted keys and writes, the float64 oracle."""
import importlib.util
import os
import sys

import numpy as np

from pibidra_util import bf16_values, rel_rms, w64  # noqa: F401

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def oracle():
    name = "kegasun_oracle"
    if name in sys.modules:
        return sys.modules[name]
    spec = importlib.util.spec_from_file_location(name, os.path.join(ROOT, "oracle", "kegasun_oracle.py"))
    mod = importlib.util.module_from_spec(spec)
    sys.modules[name] = mod
    spec.loader.exec_module(mod)
    return mod


def configs(S):
    """name -> config.  Sizes differ from one another on purpose: unequal head / key / value / latent sizes, sizes that are no
    multiple of 4, windows of one token, of a few, of more than the sequence, different windows in one model, layers without a
    feed-forward, all experts and one expert chosen, key sizes on every side of the matrix memory's lane rows, an odd width, a
    model without bigram rows."""
    A, M, D, X = S.kegasun_attention, S.kegasun_mlstm, S.kegasun_dense, S.kegasun_moe
    return {
        "mixed": S.kegasun_config(64, 96, [A(4, 16, 12, 24, 20, 7, D(80)), M(3, 20, 28, X(5, 2, 24)), A(3, 12, 16, 16, 28, 19, X(4, 1, 40)), M(2, 16, 16, D(48), gate_cap=6.0)]),
        "odd": S.kegasun_config(37, 51, [M(2, 7, 5, None, gate_cap=3.0), A(5, 5, 9, 11, 13, 3, X(3, 3, 10)), A(1, 9, 3, 5, 7, 300, D(21), scale=0.9), M(1, 1, 19, X(1, 1, 8))], eps=1e-3, bigram=(13, 29, 3)),
        "attention_only": S.kegasun_config(48, 70, [A(2, 8, 24, 40, 8, 1, D(60)), A(6, 10, 6, 12, 36, 12, None), A(3, 20, 20, 16, 16, 33, X(6, 6, 16))], scale=2.0, bigram=None),
        "memory_only": S.kegasun_config(56, 80, [M(1, 40, 33, D(60)), M(4, 17, 14, None, gate_cap=8.0), M(2, 130, 20, X(7, 3, 12)), M(3, 3, 40, None)], eps=1e-6),
        # shapes the tensor-core prefill takes: widths in whole GEMM tiles, (key, value) sizes 64 / 64, 128 / 128 and 128 / 64, latents of whole 64-column blocks, expert
        # widths of 128 (plain experts on the tcgen05 GEMM) and below
        "tiles_a": S.kegasun_config(128, 256, [A(2, 64, 64, 64, 64, 50, D(256)), M(2, 64, 64, X(4, 2, 128)), A(2, 64, 64, 128, 128, 170, X(3, 1, 64)), A(1, 64, 64, 24, 40, 90, None)], bigram=(211, 17, 6)),
        "tiles_b": S.kegasun_config(256, 384, [A(2, 128, 128, 64, 192, 77, X(6, 2, 256)), M(1, 256, 128, D(128)), A(3, 128, 64, 128, 64, 131, D(384)), A(2, 128, 128, 64, 64, 500, X(2, 2, 128))]),
    }


def decisive_routing(cfg, w, seed: int = 0):
    """Weights whose routers never face a close call, for comparisons in reduced precision (a flipped expert is a different
    function, not a rounding error).  The last R entries of the width are reserved for routing: a token's embedding holds there a
    ladder 0.5, 1, ... in an order of its own, bigram rows and all sublayers leave them alone, the sinusoid (there nearly sin 0 and
    cos 0: the slowest frequencies) is compensated, the second norm passes them with unit weight, and router row e reads one of
    them.  Everything else stays random, and all other weights read the reserved entries like any other."""
    rng = np.random.default_rng(seed)
    E, V = cfg["width"], cfg["vocab"]
    R = max([lc["mlp"]["router"]["experts"] for lc in cfg["layers"] if lc["mlp"] is not None and lc["mlp"]["kind"] == "moe"] + [1])
    w = {k: v.copy() for k, v in w.items()}
    cos_entries = (np.arange(E - R, E) % 2).astype(np.float32)
    for t in range(V):
        w["embed"][t, E - R:] = (0.5 * (1 + rng.permutation(R)) - cos_entries) / cfg["embedding"]["scale"]
    if "bigram" in w:
        w["bigram"][:, E - R:] = 0.0
    for i, lc in enumerate(cfg["layers"]):
        w[f"l{i}.mix.o"][E - R:] = 0.0
        if lc["mlp"] is None:
            continue
        for k in w:
            if k.startswith(f"l{i}.mlp.") and k.endswith("down"):
                w[k][E - R:] = 0.0
        if lc["mlp"]["kind"] != "moe":
            continue
        n = lc["mlp"]["router"]["experts"]
        r = np.zeros((n, E), dtype=np.float32)
        r[np.arange(n), E - R + rng.permutation(R)[:n]] = 4.0
        w[f"l{i}.mlp.router"] = r
        w[f"l{i}.mlp.router.b"] = (0.02 * rng.standard_normal(n)).astype(np.float32)
        w[f"l{i}.norm2"][E - R:] = 1.0
    return bf16_values(w)


def min_margin(O, cfg, w, toks):
    """Smallest gap, over all tokens and routers, between the logits of the last chosen and the first rejected expert."""
    m = []
    O.forward(cfg, w, toks, margins=m)
    return min(m) if m else np.inf


def rounding_shift(O, cfg, w, toks):
    """How far rounding the norms' outputs to BF16 (what the matrix products read in BF16 mode) alone moves a logits row of the float64
    oracle.  A read-out of the matrix memory is divided by its own size, so a row whose <n, q> nearly vanishes (above all a first token:
    one write, read along <k, q>) may turn by any amount under rounding; such rows compare nothing."""
    exact = O.layer_norm
    ref = O.forward(cfg, w, toks)
    try:
        O.layer_norm = lambda v, weight, eps: bf16_values({"v": exact(v, weight, eps)})["v"].astype(np.float64)
        got = O.forward(cfg, w, toks)
    finally:
        O.layer_norm = exact
    return max(rel_rms(got[t], ref[t]) for t in range(len(toks)))


def settled_weights(S, O, cfg, seed, toks, shift):
    """Random weights with decisive routers that rounding moves by at most `shift` (the first of the seeds from `seed` on)."""
    for k in range(seed, seed + 40):
        w = decisive_routing(cfg, S.kegasun_weights(cfg, k), k)
        if min_margin(O, cfg, w64(w), toks) > 0.15 and rounding_shift(O, cfg, w64(w), toks) <= shift:
            return w
    raise AssertionError("no seed gives a well-conditioned model")


def _one_hot_model(S, layer, V: int, E: int, seed: int, bigram=None, eps: float = 1e-5):
    """One layer over one-hot embeddings that stand out of the sinusoid (entries of 40 against 1)."""
    cfg = S.kegasun_config(E, V, [layer], eps=eps, scale=40.0, bigram=bigram)
    w = S.kegasun_weights(cfg, seed)
    emb = np.zeros((V, E), dtype=np.float32)
    emb[np.arange(V), np.arange(V)] = 1.0
    w["embed"] = emb
    w["l0.norm1"][:] = 1.0
    return cfg, w


def needle_attention(S, window: int, key_dim: int = 8, value_dim: int = 12, seed: int = 3):
    """One attention layer decided by ONE planted key: the query latent of token A and the latent of token B are aligned through
    rank-one W_uq and W_uk, the latents of all other tokens have no part along B's direction, and B's value is large.  Returns
    (config, weights, A, B, filler tokens)."""
    E, V, H, Rq, R = 64, 48, 3, 16, 32
    cfg, w = _one_hot_model(S, S.kegasun_attention(H, key_dim, value_dim, Rq, R, window, None, scale=1.0), V, E, seed)
    rng = np.random.default_rng(seed)
    A, B = 5, 9

    def unit(n):
        v = rng.standard_normal(n)
        return (v / np.linalg.norm(v)).astype(np.float32)

    a, b = unit(Rq), unit(R)
    w["l0.mix.dq.norm"][:] = 1.0
    w["l0.mix.dkv.norm"][:] = 1.0
    w["l0.mix.dq"] -= np.outer(a, a @ w["l0.mix.dq"])
    w["l0.mix.dkv"] -= np.outer(b, b @ w["l0.mix.dkv"])
    w["l0.mix.dq"][:, A] = 3.0 * a
    w["l0.mix.dkv"][:, B] = 3.0 * b
    for h in range(H):
        u = unit(key_dim)
        w["l0.mix.uq"][h * key_dim:(h + 1) * key_dim] = np.outer(u, a)
        w["l0.mix.uk"][h * key_dim:(h + 1) * key_dim] = 0.6 * np.outer(u, b)  # e_AB = 0.6 sqrt(Rq R) = 13.6
    w["l0.mix.uv"] += 1.5 * np.outer(rng.standard_normal(H * value_dim), b).astype(np.float32)
    w["l0.mix.sink"][:] = 1.0
    w["l0.mix.g"][:, A] = 0.5
    fill = [t for t in range(V) if t not in (A, B)]
    return cfg, bf16_values(w), A, B, fill


def needle_mlstm(S, key_dim: int = 12, value_dim: int = 10, seed: int = 4):
    """One matrix memory that keeps what tokens B and C wrote along the same key: forget gates of (nearly) one, fillers whose keys
    are zero; the read-out at A is the mean of both values, so losing either write turns its direction (the normaliser makes its
    size meaningless).  Returns (config, weights, A, B, C, filler tokens)."""
    E, V, H = 64, 48, 2
    cfg, w = _one_hot_model(S, S.kegasun_mlstm(H, key_dim, value_dim, None, gate_cap=14.0), V, E, seed)
    rng = np.random.default_rng(seed)
    A, B, C = 5, 9, 21
    u = rng.standard_normal(H * key_dim).astype(np.float32)
    w["l0.mix.f"][:] = 0.0
    w["l0.mix.f.b"][:] = 12.0   # log forget gate -2e-5 per token behind the cap
    w["l0.mix.i"][:] = 0.0
    w["l0.mix.i.b"][:] = 0.0
    w["l0.mix.k"][:] = 0.0
    w["l0.mix.k"][:, B] = u
    w["l0.mix.k"][:, C] = u
    w["l0.mix.q"][:, A] = u
    w["l0.mix.v"][:, B] = rng.standard_normal(H * value_dim).astype(np.float32)
    w["l0.mix.v"][:, C] = rng.standard_normal(H * value_dim).astype(np.float32)
    w["l0.mix.g"][:, A] = 0.5
    w["l0.mix.o"] *= 4.0      # against the one-hot embedding of A
    fill = [t for t in range(V) if t not in (A, B, C)]
    return cfg, bf16_values(w), A, B, C, fill


def random_layer_list(S, rng, wide: bool = False):
    """A random list of 1 .. 6 layers with random sizes and constants; wide: sizes that take the tensor-core kernels."""
    layers = []
    for _ in range(int(rng.integers(1, 7))):
        pick = rng.random()
        if rng.random() < 0.2:
            mlp = None
        elif rng.random() < 0.5:
            mlp = S.kegasun_dense(int(rng.choice([64, 128, 256])) if wide else int(rng.integers(4, 70)))
        else:
            X = int(rng.integers(1, 9))
            mlp = S.kegasun_moe(X, int(rng.integers(1, X + 1)), int(rng.choice([64, 128])) if wide else int(rng.integers(3, 40)))
        if pick < 0.55:
            if wide:
                dk, dv = [(64, 64), (128, 128), (128, 64), (32, 32)][int(rng.integers(0, 4))]
                layers.append(S.kegasun_attention(int(rng.choice([1, 2, 4])), dk, dv, int(rng.choice([48, 64, 128])), int(rng.choice([40, 64, 128])), int(rng.choice([9, 64, 65, 128, 400])), mlp))
            else:
                dk = int(rng.integers(1, 30))
                layers.append(S.kegasun_attention(int(rng.integers(1, 7)), dk, int(rng.integers(1, 40)), int(rng.integers(2, 40)), int(rng.integers(2, 50)), int(rng.choice([1, 2, 5, 16, 31, 64, 200])), mlp,
                                                  scale=float(rng.uniform(0.3, 2.0)) * dk ** -0.5))
        else:
            dk = int(rng.choice([16, 32, 64, 128])) if wide else int(rng.integers(1, 60))
            layers.append(S.kegasun_mlstm(int(rng.integers(1, 5)), dk, int(rng.choice([16, 64, 100])) if wide else int(rng.integers(1, 40)), mlp, gate_cap=float(rng.uniform(1.0, 20.0))))
    return layers
