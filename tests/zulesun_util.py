"""Shared helpers of the Zulesun tests: small configurations, weights with planted keys and writes, the float64 oracle."""
import importlib.util
import os
import sys

import numpy as np

from pibidra_util import bf16_values, rel_rms, w64  # noqa: F401

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def oracle():
    name = "zulesun_oracle"
    if name in sys.modules:
        return sys.modules[name]
    spec = importlib.util.spec_from_file_location(name, os.path.join(ROOT, "oracle", "zulesun_oracle.py"))
    mod = importlib.util.module_from_spec(spec)
    sys.modules[name] = mod
    spec.loader.exec_module(mod)
    return mod


def configs(S):
    """name -> config.  Sizes differ from one another on purpose: unequal head / key / value / state sizes, grouped and ungrouped
    key/value heads, sizes that are no multiple of 4, chunks of one token, of a few, of more than the sequence, different chunks in one
    model, layers without a feed-forward, one and all experts chosen, one group and several, an odd width, a model without a token
    input."""
    P, L, D, X = S.zulesun_parallel, S.zulesun_lightning, S.zulesun_dense, S.zulesun_moe
    return {
        "mixed": S.zulesun_config(64, 96, [P(4, 2, 16, 12, 7, 40, 6, 5, 4, D(80)), L(3, 20, 28, X(6, 2, 24, 3, 2)), P(3, 3, 12, 16, 19, 56, 16, 8, 3, X(4, 1, 40)), L(2, 16, 16, D(48), decay=[0.5, 0.995])]),
        "odd": S.zulesun_config(37, 51, [L(2, 7, 5, None), P(5, 1, 6, 9, 3, 13, 3, 1, 2, X(3, 3, 10)), P(1, 1, 9, 3, 300, 7, 1, 3, 5, D(21), scale=0.9, factor=None, softcap=3.0), L(1, 1, 19, X(2, 1, 8, 2, 1))],
                              side=5, eps=1e-3, scale=2.5),
        "parallel_only": S.zulesun_config(48, 70, [P(2, 1, 8, 24, 1, 24, 20, 4, 4, D(60)), P(6, 2, 10, 6, 12, 30, 8, 6, 1, None, rot_dims=10), P(3, 1, 20, 20, 33, 64, 33, 7, 6, X(6, 6, 16, 2, 2), rot_dims=2)], side=None),
        "lightning_only": S.zulesun_config(56, 80, [L(1, 40, 33, D(60)), L(4, 17, 14, None), L(2, 130, 20, X(8, 3, 12, 4, 2)), L(3, 3, 40, None)], side=7, eps=1e-6),
        # shapes the tensor-core prefill takes: widths in whole GEMM tiles, (key, value) sizes 64 / 64, 64 / 32, 128 / 128 and 128 / 64, scan channels and step ranks of
        # whole 64-column blocks, expert widths of 64 and 128, token inputs in whole blocks
        "tiles_a": S.zulesun_config(128, 256, [P(2, 1, 64, 64, 50, 128, 16, 64, 4, D(256)), L(2, 64, 64, X(4, 2, 128, 2, 1)), P(4, 2, 64, 32, 96, 192, 32, 64, 3, X(3, 1, 64)), L(1, 128, 64, None)], side=64),
        "tiles_b": S.zulesun_config(256, 384, [P(2, 2, 128, 128, 77, 256, 8, 128, 4, X(6, 2, 256, 3, 2)), L(2, 128, 128, D(128)), P(2, 1, 128, 64, 131, 128, 12, 16, 2, D(384)), L(4, 32, 192, X(2, 2, 128))], side=128),
    }


def routers(cfg):
    return [(i, lc["mlp"]["router"]) for i, lc in enumerate(cfg["layers"]) if lc["mlp"] is not None and lc["mlp"]["kind"] == "moe"]


def decisive_routing(cfg, w, seed: int = 0):
    """Weights whose routers never face a close call, for comparisons in reduced precision (a flipped expert is a different
    function, not a rounding error).  The last R entries of the width are reserved for routing: a token's embedding holds there a
    ladder 0.5, 1, ... in an order of its own, all sublayers leave them alone, the second norm passes them with unit weight, and router
    row e reads one of them (so experts and groups are told apart by steps of the ladder).  Everything else stays random, and all other
    weights read the reserved entries like any other."""
    rng = np.random.default_rng(seed)
    E, V = cfg["width"], cfg["vocab"]
    R = max([r["experts"] for _, r in routers(cfg)] + [1])
    w = {k: v.copy() for k, v in w.items()}
    for t in range(V):
        w["embed"][t, E - R:] = 0.5 * (1 + rng.permutation(R)) / cfg["embedding"]["scale"]
    for i, lc in enumerate(cfg["layers"]):
        w[f"l{i}.norm1b"][E - R:] = -1.0
        if lc["mlp"] is not None:
            w[f"l{i}.norm2b"][E - R:] = -1.0
        if cfg.get("token_side"):
            w[f"l{i}.side.norm"][E - R:] = 0.0
    for i, r in routers(cfg):
        n = r["experts"]
        m = np.zeros((n, E), dtype=np.float32)
        m[np.arange(n), E - R + rng.permutation(R)[:n]] = 4.0
        w[f"l{i}.mlp.router"] = m
        w[f"l{i}.norm2"][E - R:] = 0.0
    return bf16_values(w)


def min_margin(O, cfg, w, toks):
    """Smallest gap, over all tokens and routers, between what was chosen and what was not (groups and experts)."""
    m = []
    O.forward(cfg, w, toks, margins=m)
    return min(m) if m else np.inf


def rounding_shift(O, cfg, w, toks, bits: int = 9):
    """How far disturbing what the weight matrices read by up to 2^-bits alone moves a logits row of the float64 oracle: three random disturbances
    and, for the 9 bits of BF16, the rounding itself.  Read-outs that are divided by their own size turn by any amount where <k, q> or a scan's
    result nearly vanishes (above all at first tokens); such rows compare nothing."""
    exact = O.linear
    ref = O.forward(cfg, w, toks)
    rng = np.random.default_rng(0)
    worst = 0.0
    try:
        for k in range(0 if bits == 9 else 1, 4):
            if k == 0:
                O.linear = lambda x, m: exact(bf16_values({"x": x})["x"].astype(np.float64), m)
            else:
                O.linear = lambda x, m: exact(x * (1.0 + 2.0 ** -bits * rng.uniform(-1.0, 1.0, x.shape)), m)
            got = O.forward(cfg, w, toks)
            worst = max(worst, max(rel_rms(got[t], ref[t]) for t in range(len(toks))))
    finally:
        O.linear = exact
    return worst


def settled_weights(S, O, cfg, seed, toks, shift):
    """Random weights with decisive routers that rounding moves by at most `shift` (the first of the seeds from `seed` on)."""
    for k in range(seed, seed + 40):
        w = decisive_routing(cfg, S.zulesun_weights(cfg, k), k)
        if min_margin(O, cfg, w64(w), toks) > 0.15 and rounding_shift(O, cfg, w64(w), toks) <= shift:
            return w
    raise AssertionError("no seed gives a well-conditioned model")


def _one_hot_model(S, layer, V: int, E: int, seed: int, eps: float = 1e-5):
    """One layer over one-hot embeddings (small against the layer's contribution), no token input."""
    cfg = S.zulesun_config(E, V, [layer], side=None, eps=eps, scale=2.0)
    w = S.zulesun_weights(cfg, seed)
    emb = np.zeros((V, E), dtype=np.float32)
    emb[np.arange(V), np.arange(V)] = 1.0
    w["embed"] = emb
    w["l0.norm1"][:] = 0.0
    w["l0.norm1b"][:] = 0.0
    return cfg, w


def needle_chunk(S, chunk: int, key_dim: int = 8, value_dim: int = 12, seed: int = 3):
    """One parallel layer (the scan's part weighted with zero) decided by ONE planted key: the query of token A and the key of token B lie
    along one direction of the unrotated entries, the keys of all other tokens have no part along it, and B's value is large.  Returns
    (config, weights, A, B, filler tokens)."""
    E, V, H, G = 64, 48, 4, 2
    rot = 2
    cfg, w = _one_hot_model(S, S.zulesun_parallel(H, G, key_dim, value_dim, chunk, 8, 4, 2, 3, None, rot_dims=rot, scale=16.0 / key_dim, softcap=40.0, branch_scale=(1.0, 0.0)), V, E, seed)
    rng = np.random.default_rng(seed)
    A, B = 5, 9
    q = "l0.mix.left."
    w[q + "q.norm"][:], w[q + "k.norm"][:] = 1.0, 1.0
    for g in range(G):
        u = np.zeros(key_dim, dtype=np.float32)
        u[rot:] = rng.standard_normal(key_dim - rot)
        u /= np.linalg.norm(u)
        rows = slice(g * key_dim, (g + 1) * key_dim)
        w[q + "k"][rows] -= np.outer(u, u @ w[q + "k"][rows])
        w[q + "k"][rows, B] = 3.0 * u
        for h in range(g * H // G, (g + 1) * H // G):
            w[q + "q"][h * key_dim:(h + 1) * key_dim, A] = 3.0 * u
    w[q + "v"][:, B] *= 4.0
    w[q + "g"][:, A] = 0.5
    fill = [t for t in range(V) if t not in (A, B)]
    return cfg, bf16_values(w), A, B, fill


def needle_lightning(S, key_dim: int = 12, value_dim: int = 10, seed: int = 4):
    """One decayed linear attention that keeps what tokens B and C wrote along the same key: decays near one, fillers whose keys are
    zero; the read-out at A is a mean of both values, so losing either write turns its direction (the norm makes its size meaningless).
    Returns (config, weights, A, B, C, filler tokens)."""
    E, V, H = 64, 48, 2
    cfg, w = _one_hot_model(S, S.zulesun_lightning(H, key_dim, value_dim, None, decay=[0.9995, 0.999]), V, E, seed)
    rng = np.random.default_rng(seed)
    A, B, C = 5, 9, 21
    u = np.abs(rng.standard_normal(H * key_dim)).astype(np.float32)
    w["l0.mix.k"][:] = 0.0
    w["l0.mix.k"][:, B] = u
    w["l0.mix.k"][:, C] = u
    w["l0.mix.q"][:, A] = u
    w["l0.mix.v"][:, B] = rng.standard_normal(H * value_dim).astype(np.float32)
    w["l0.mix.v"][:, C] = rng.standard_normal(H * value_dim).astype(np.float32)
    w["l0.mix.g"][:, A] = 0.5
    fill = [t for t in range(V) if t not in (A, B, C)]
    return cfg, bf16_values(w), A, B, C, fill


def needle_scan(S, state: int = 5, taps: int = 3, seed: int = 6):
    """One parallel layer (the attention's part weighted with zero) whose scan keeps what token B wrote: fillers put nothing into the channels,
    the states barely decay, A reads what is there.  Returns (config, weights, A, B, filler tokens)."""
    E, V, I = 64, 48, 24
    cfg, w = _one_hot_model(S, S.zulesun_parallel(2, 1, 4, 4, 5, I, state, 3, taps, None, branch_scale=(0.0, 1.0)), V, E, seed)
    rng = np.random.default_rng(seed)
    A, B = 5, 9
    r = "l0.mix.right."
    w[r + "in"][:I] = 0.0
    w[r + "in"][:I, A] = 0.15 * rng.standard_normal(I)
    w[r + "in"][:I, B] = 0.8 * rng.standard_normal(I)
    w[r + "conv.b"][:] = 0.0
    w[r + "A_log"][:] = -8.0 + 0.5 * rng.standard_normal((I, state))
    w[r + "D"][:] = 0.1
    w[r + "dt.b"][:] = -0.5
    fill = [t for t in range(V) if t not in (A, B)]
    return cfg, bf16_values(w), A, B, fill


def random_layer_list(S, rng, wide: bool = False):
    """A random list of 1 .. 5 layers with random sizes and constants; wide: sizes that take the tensor-core kernels."""
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        if rng.random() < 0.2:
            mlp = None
        elif rng.random() < 0.4:
            mlp = S.zulesun_dense(int(rng.choice([64, 128, 256])) if wide else int(rng.integers(4, 70)))
        else:
            groups, per = int(rng.integers(1, 4)), int(rng.integers(1, 4))
            keep = int(rng.integers(1, groups + 1))
            mlp = S.zulesun_moe(groups * per, int(rng.integers(1, keep * per + 1)), int(rng.choice([64, 128])) if wide else int(rng.integers(3, 40)), groups, keep)
        if rng.random() < 0.6:
            G = int(rng.integers(1, 4))
            if wide:
                dk, dv = [(64, 64), (128, 128), (128, 64), (64, 32), (32, 32)][int(rng.integers(0, 5))]
                layers.append(S.zulesun_parallel(G * int(rng.integers(1, 3)), G, dk, dv, int(rng.choice([9, 64, 65, 128, 400])), int(rng.choice([64, 128, 320])), int(rng.choice([4, 16, 32, 64])),
                                                 int(rng.choice([8, 64, 128])), int(rng.integers(1, 6)), mlp, rot_dims=int(rng.choice([16, 32]))))
            else:
                dk = int(rng.integers(1, 30))
                layers.append(S.zulesun_parallel(G * int(rng.integers(1, 4)), G, dk, int(rng.integers(1, 40)), int(rng.choice([1, 2, 5, 16, 31, 64, 200])), int(rng.integers(1, 90)), int(rng.integers(1, 40)),
                                                 int(rng.integers(1, 12)), int(rng.integers(1, 7)), mlp, rot_dims=2 * int(rng.integers(0, dk // 2 + 1)), base=float(rng.choice([100.0, 10000.0])),
                                                 factor=None if rng.random() < 0.3 else float(rng.uniform(0.5, 16.0)), scale=float(rng.uniform(0.3, 2.0)) * dk ** -0.5, softcap=float(rng.uniform(2.0, 50.0)),
                                                 branch_scale=(float(rng.uniform(0.2, 1.5)), float(rng.uniform(0.2, 1.5)))))
        else:
            H = int(rng.integers(1, 5))
            dk = int(rng.choice([32, 64, 128])) if wide else int(rng.integers(1, 60))
            layers.append(S.zulesun_lightning(H, dk, int(rng.choice([16, 64, 100])) if wide else int(rng.integers(1, 40)), mlp, decay=rng.uniform(0.3, 0.9999, H).tolist()))
    return layers
