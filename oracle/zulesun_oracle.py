"""Plain float64 restatement of the Zulesun forward pass (test infrastructure only).

One function per mechanism, no cache, no state object, no batching: every call recomputes the whole sequence, attention runs over full
score matrices, both recurrences run token by token in explicit loops.  The product path never imports this file.

Notation.  x[t] is the residual row of token t (width E).  R(v; w) = v / sqrt(mean v^2 + eps) * w,  N(v; w) = R(v; 1 + w).
    x[t] = scale * embed[token_t]
    x <- x + N(mixer(N(x; norm1)); norm1b);   x <- x + N(ff(N(x; norm2)); norm2b)  (when the layer has a feed-forward)
    x <- x + R(P (gelu_tanh(G x) * e_i); side.norm),  e_i[t] = entries [i D, (i + 1) D) of side.embed[token_t] for layer i
    logits = head N(x; final.norm)

Mixer "lightning" (H heads, key size d, value size dv, decay c_a per head):
    q = silu(Wq h), k = silu(Wk h) as [H][d];   v = silu(Wv h) as [H][dv];   S <- c_a S + k v^T (from zero),  o = S^T q
    out = Wo (R(concat_a o^a; norm) * sigmoid(Wg h))     (ONE statistic over all heads)

Mixer "parallel": left_scale * attention(h) + right_scale * mamba(h).
  attention (H query heads, G key/value heads, key size d, value size dv, chunk size C):
    q = R(Wq h; q.norm), k = R(Wk h; k.norm) (one statistic over all heads), then the first `dims` entries of every head turn:
    pair (i, i + dims/2) by the angle p * base^(-2i/dims) / factor;   v = Wv h
    e_ij = cap tanh(s <q_i, k_j> / cap)  for j <= i in the same chunk (i div C = j div C);  softmax;  o_i = sum_j p_ij v_j
    out = Wo (concat o * sigmoid(Wg h))
  mamba (I channels, N states per channel, rank Rd, K taps):
    [x | z] = Win h;   x = silu(conv(x) + b) per channel, last tap = the current token;   [dt | B | C] = Wx x
    dt = softplus(Wdt dt + dt.b);   S[c, n] <- exp(-exp(A_log[c, n]) dt_c) S[c, n] + dt_c x_c B_n (from zero);   y_c = <S[c], C> + D_c x_c
    out = Wo (y * silu(z))

Feed-forward "dense": Wdown relu(Wup h)^2.
Feed-forward "moe": s = softmax(Wrouter h); the experts form `count` equal groups of neighbours, a group scores the largest s in it, only
experts of the `keep` best groups compete; the `top` largest s of them; out = sum_e s_e Wdown^e (silu(Wgate^e h) * (Wup^e h)).
"""
from __future__ import annotations

import json
import math
import struct

import numpy as np


def read_safetensors(path: str) -> dict:
    """name -> float64 array (BF16 / F32 widened exactly; I32 as int64)."""
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, m in head.items():
        if name == "__metadata__":
            continue
        lo, hi = m["data_offsets"]
        raw = blob[lo:hi]
        if m["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif m["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif m["dtype"] == "I32":
            a = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(f"{name}: dtype {m['dtype']}")
        out[name] = a.reshape(m["shape"])
    return out


# ---- products ----------------------------------------------------------------------------------------------------------
def linear(x, w):
    """Every product with a weight matrix [out][in] goes through here."""
    return x @ w.T


# ---- elementwise -------------------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ---- norms -------------------------------------------------------------------------------------------------------------
def rms_norm(v, w, eps: float):
    return v / np.sqrt((v * v).mean(-1, keepdims=True) + eps) * w


def block_norm(v, w, eps: float):
    """The blocks' norm: weights are stored as deviations from one."""
    return rms_norm(v, 1.0 + w, eps)


# ---- lightning attention -----------------------------------------------------------------------------------------------
def lightning_scan(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H] -> read-outs [T, H, dv]."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for a in range(H):
        S = np.zeros((d, v.shape[2]))
        for t in range(T):
            S = float(decay[a]) * S + np.outer(k[t, a], v[t, a])
            out[t, a] = S.T @ q[t, a]
    return out


def mixer_lightning(h, w: dict, pre: str, m: dict, eps: float):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(linear(h, w[pre + "q"])).reshape(T, H, d)
    k = silu(linear(h, w[pre + "k"])).reshape(T, H, d)
    v = silu(linear(h, w[pre + "v"])).reshape(T, H, dv)
    o = lightning_scan(q, k, v, m["decay"]).reshape(T, H * dv)
    return linear(rms_norm(o, w[pre + "norm"], eps) * sigmoid(linear(h, w[pre + "g"])), w[pre + "o"])


# ---- chunked attention -------------------------------------------------------------------------------------------------
def rotate_half(x, rot: dict):
    """x [T, heads, d]: the first `dims` entries of every head turned by the position's angles."""
    dims = int(rot["dims"])
    half = dims // 2
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    f = float(rot["base"]) ** (-2.0 * np.arange(half) / dims) / factor if half else np.zeros(0)
    a = np.arange(x.shape[0], dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(a)[:, None, :], np.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def chunk_mask(T: int, size: int):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def masked_softmax(e, mask):
    e = np.where(mask, e, -np.inf)
    p = np.exp(e - e.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def chunked_attention(h, w: dict, pre: str, m: dict, eps: float):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate_half(rms_norm(linear(h, w[pre + "q"]), w[pre + "q.norm"], eps).reshape(T, H, d), m["rot"])
    k = rotate_half(rms_norm(linear(h, w[pre + "k"]), w[pre + "k.norm"], eps).reshape(T, G, d), m["rot"])
    v = linear(h, w[pre + "v"]).reshape(T, G, dv)
    mask = chunk_mask(T, int(m["mask"]["size"]))
    o = np.zeros((T, H, dv))
    for a in range(H):
        g = a // (H // G)
        e = soft_cap((q[:, a] @ k[:, g].T) * float(m["scale"]), m.get("softcap"))
        o[:, a] = masked_softmax(e, mask) @ v[:, g]
    return linear(o.reshape(T, H * dv) * sigmoid(linear(h, w[pre + "g"])), w[pre + "o"])


# ---- selective scan ----------------------------------------------------------------------------------------------------
def causal_conv(x, taps, bias):
    """x [T, C], taps [C, K] (the last column meets the current token), zeros before the start."""
    K = taps.shape[1]
    xp = np.concatenate([np.zeros((K - 1, x.shape[1])), x])
    return sum(xp[i:i + x.shape[0]] * taps[:, i] for i in range(K)) + bias


def selective_scan(x, dt, B, C, A, D):
    """x, dt [T, I], B, C [T, N], A [I, N], D [I] -> y [T, I]."""
    S = np.zeros(A.shape)
    out = np.zeros(x.shape)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba(h, w: dict, pre: str, m: dict):
    inner, N, rank = int(m["inner"]), int(m["state"]), int(m["dt_rank"])
    xz = linear(h, w[pre + "in"])
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[pre + "conv"], w[pre + "conv.b"]))
    p = linear(x, w[pre + "x"])
    dt = softplus(linear(p[:, :rank], w[pre + "dt"]) + w[pre + "dt.b"])
    y = selective_scan(x, dt, p[:, rank:rank + N], p[:, rank + N:], -np.exp(w[pre + "A_log"]), w[pre + "D"])
    return linear(y * silu(z), w[pre + "o"])


def mixer_parallel(h, w: dict, pre: str, m: dict, eps: float):
    return float(m["left_scale"]) * chunked_attention(h, w, pre + "left.", m["left"], eps) + float(m["right_scale"]) * mamba(h, w, pre + "right.", m["right"])


# ---- feed-forward ------------------------------------------------------------------------------------------------------
def ff_dense(h, w: dict, pre: str):
    return linear(np.maximum(linear(h, w[pre + "up"]), 0.0) ** 2, w[pre + "down"])


def expert(h, w: dict, pre: str):
    return linear(silu(linear(h, w[pre + "gate"])) * linear(h, w[pre + "up"]), w[pre + "down"])


def moe_route(h, w: dict, pre: str, router: dict, margins=None):
    """(ids [T, top], weights [T, top]); margins (a list) receives, per token, the smaller of the two gaps that decide, in logits: between
    the worst kept and the best dropped group, and between the last chosen and the first rejected expert of the kept groups."""
    z = linear(h, w[pre + "router"])
    s = np.exp(z - z.max(-1, keepdims=True))
    s /= s.sum(-1, keepdims=True)
    T, X = s.shape
    gr = router.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = int(gr["count"]), int(gr["keep"]), int(router["top"])
    per = X // count
    ids = np.zeros((T, top), dtype=np.int64)
    for t in range(T):
        best = s[t].reshape(count, per).max(-1)
        order = np.argsort(-best, kind="stable")
        kept = set(order[:keep].tolist())
        can = np.array([e for e in range(X) if e // per in kept])
        pick = can[np.argsort(-s[t][can], kind="stable")]
        ids[t] = pick[:top]
        if margins is not None:
            zg = z[t].reshape(count, per).max(-1)
            gaps = []
            if keep < count:
                gaps.append(zg[order[keep - 1]] - zg[order[keep]])
            if top < len(pick):
                gaps.append(z[t][pick[top - 1]] - z[t][pick[top]])
            margins.extend([min(gaps)] if gaps else [])
    return ids, np.take_along_axis(s, ids, -1)


def ff_moe(h, w: dict, pre: str, mlp: dict, margins=None):
    ids, wts = moe_route(h, w, pre, mlp["router"], margins)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t], wts[t]):
            out[t] += wt * expert(h[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


# ---- per-layer token input ---------------------------------------------------------------------------------------------
def token_side(x, tokens, w: dict, pre: str, layer: int, dim: int, eps: float):
    e = w["side.embed"][np.asarray(tokens)][:, layer * dim:(layer + 1) * dim]
    y = linear(gelu_tanh(linear(x, w[pre + "side.gate"])) * e, w[pre + "side.proj"])
    return rms_norm(y, w[pre + "side.norm"], eps)


# ---- model -------------------------------------------------------------------------------------------------------------
MIXERS = {"lightning": mixer_lightning, "parallel": mixer_parallel}


def forward(cfg: dict, w: dict, tokens, return_layers: bool = False, margins=None):
    """Logits [T, vocab] of the whole sequence (and, optionally, the residual stream after every layer [layers, T, E])."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    trace = []
    for i, lc in enumerate(cfg["layers"]):
        pre = f"l{i}."
        y = MIXERS[lc["type"]](block_norm(x, w[pre + "norm1"], eps), w, pre + "mix.", lc["mixer"], eps)
        x = x + block_norm(y, w[pre + "norm1b"], eps)
        mlp = lc.get("mlp")
        if mlp is not None:
            h = block_norm(x, w[pre + "norm2"], eps)
            y = ff_dense(h, w, pre + "mlp.") if mlp["kind"] == "dense" else ff_moe(h, w, pre + "mlp.", mlp, margins)
            x = x + block_norm(y, w[pre + "norm2b"], eps)
        if cfg.get("token_side"):
            x = x + token_side(x, tokens, w, pre, i, int(cfg["token_side"]["dim"]), eps)
        trace.append(x.copy())
    logits = linear(block_norm(x, w["final.norm"], eps), w["head"])
    return (logits, np.stack(trace)) if return_layers else logits


def load_dir(path: str):
    with open(f"{path}/config.json") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(f"{path}/model.safetensors")
