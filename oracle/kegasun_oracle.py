"""Plain float64 restatement of the Kegasun forward pass (test infrastructure only).

One function per mechanism, no cache, no state object, no batching: every call recomputes the whole sequence, keys and values are
expanded per head from the latent, the matrix memory runs token by token in an explicit loop.  The product path never imports
this file.

Notation.  x[t] is the residual row of token t (width E).  LN(v; w) = (v - mean v) / sqrt(mean (v - mean v)^2 + eps) * w,
RN(v; w) = v / sqrt(mean v^2 + eps) * w.
    x[t] = scale * embed[token_t] + bigram[b_t] + P(t)
        b_t = (mul_prev * token_(t-1) + mul_cur * token_t) mod buckets, b_0 = buckets
        P(t)[2i] = sin(t * 10000^(-2i/E)),  P(t)[2i+1] = cos(t * 10000^(-2i/E))
    x <- x + mixer(LN(x; norm1));   x <- x + ff(LN(x; norm2))  (when the layer has a feed-forward);   logits = head LN(x; final.norm)

Mixer "latent_attention" (H heads, key size d, value size dv, query latent of rank Rq, key/value latent of rank R, window W):
    q = Wuq RN(Wdq h; dq.norm) as [H][d];   c = RN(Wdkv h; dkv.norm);   k_j^a = Wuk^a c_j,  v_j^a = Wuv^a c_j
    e_ij = s <q_i, k_j>  for 0 <= i - j < W;   p_ij = exp(e_ij) / (exp(z_a) + sum_j exp(e_ij))   (z_a: the head's sink)
    o_i^a = sigmoid(<Wg_a, h_i>) sum_j p_ij v_j^a;   out = Wo concat_a o^a

Mixer "mlstm" (H heads, key size d, value size dv, cap C):
    q = Wq h / sqrt(d),  k = Wk h  as [H][d];   v = Wv h as [H][dv]
    i = C tanh((<Wi_a, h> + bi_a) / C);   f = log sigmoid(C tanh((<Wf_a, h> + bf_a) / C))
    m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n <- exp(f + m - m') n + exp(i - m') k;  m <- m'  (all from zero)
    o = S^T q / (max(|<n, q>|, exp(-m)) + 1e-6);   per head o / sqrt(mean o^2 + eps);   out = Wo (concat_a o^a * norm * sigmoid(Wg h))

Feed-forward "dense": Wdown (silu(Wgate h) * (Wup h)).
Feed-forward "moe": z = Wrouter h + b; the `top` largest z are chosen, weights = softmax over the chosen z;
    out = sum_e w_e Wdown^e relu(Wup^e h)^2.
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


# ---- elementwise -------------------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def silu(z):
    return z * sigmoid(z)


def relu_squared(z):
    return np.maximum(z, 0.0) ** 2


def soft_cap(z, cap: float):
    return cap * np.tanh(z / cap)


# ---- norms -------------------------------------------------------------------------------------------------------------
def layer_norm(v, w, eps: float):
    d = v - v.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w


def rms_norm(v, w, eps: float):
    out = v / np.sqrt((v * v).mean(-1, keepdims=True) + eps)
    return out if w is None else out * w


# ---- embedding ---------------------------------------------------------------------------------------------------------
def bigram_rows(tokens, bg: dict):
    t = [int(v) for v in tokens]
    return [int(bg["buckets"]) if p == 0 else (t[p - 1] * int(bg["mul_prev"]) + t[p] * int(bg["mul_cur"])) % int(bg["buckets"]) for p in range(len(t))]


def sinusoid(T: int, width: int):
    out = np.zeros((T, width))
    for e in range(width):
        f = 10000.0 ** (-2.0 * (e // 2) / width)
        out[:, e] = (np.cos if e % 2 else np.sin)(np.arange(T, dtype=np.float64) * f)
    return out


def embedding(cfg: dict, w: dict, tokens):
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    if cfg["embedding"].get("bigram"):
        x = x + w["bigram"][bigram_rows(tokens, cfg["embedding"]["bigram"])]
    return x + sinusoid(len(tokens), int(cfg["width"]))


# ---- latent attention --------------------------------------------------------------------------------------------------
def window_mask(T: int, window: int):
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < window)


def sink_softmax(e, mask, sink: float):
    """e, mask [T, T]: weights of the visible keys with exp(sink) as one more term of the denominator."""
    e = np.where(mask, e, -np.inf)
    mx = np.maximum(e.max(-1, keepdims=True), sink)
    p = np.exp(e - mx)
    return p / (p.sum(-1, keepdims=True) + np.exp(sink - mx))


def mixer_latent_attention(h, w: dict, pre: str, m: dict, eps: float):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    cq = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps)
    q = (cq @ w[pre + "uq"].T).reshape(T, H, d)
    c = rms_norm(h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], eps)
    k = (c @ w[pre + "uk"].T).reshape(T, H, d)
    v = (c @ w[pre + "uv"].T).reshape(T, H, dv)
    gate = sigmoid(h @ w[pre + "g"].T)
    mask = window_mask(T, int(m["mask"]["size"]))
    o = np.zeros((T, H, dv))
    for a in range(H):
        p = sink_softmax((q[:, a] @ k[:, a].T) * float(m["scale"]), mask, float(w[pre + "sink"][a]))
        o[:, a] = (p @ v[:, a]) * gate[:, a:a + 1]
    return o.reshape(T, H * dv) @ w[pre + "o"].T


# ---- matrix memory -----------------------------------------------------------------------------------------------------
def mlstm_gates(h, w: dict, pre: str, cap: float):
    """(log input gate, log forget gate) [T, H]."""
    i = soft_cap(h @ w[pre + "i"].T + w[pre + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[pre + "f"].T + w[pre + "f.b"], cap))
    return i, f


def mlstm_scan(q, k, v, i, f):
    """q, k [T, H, d] (q scaled), v [T, H, dv], i, f [T, H] -> read-outs [T, H, dv]."""
    T, H, d = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for a in range(H):
        S, n, m = np.zeros((d, v.shape[2])), np.zeros(d), 0.0
        for t in range(T):
            m1 = max(f[t, a] + m, i[t, a])
            keep, write = math.exp(f[t, a] + m - m1), math.exp(i[t, a] - m1)
            S = keep * S + write * np.outer(k[t, a], v[t, a])
            n = keep * n + write * k[t, a]
            m = m1
            out[t, a] = (S.T @ q[t, a]) / (max(abs(float(n @ q[t, a])), math.exp(-m)) + 1e-6)
    return out


def mixer_mlstm(h, w: dict, pre: str, m: dict, eps: float):
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[pre + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, d)
    v = (h @ w[pre + "v"].T).reshape(T, H, dv)
    i, f = mlstm_gates(h, w, pre, float(m["gate_cap"]))
    o = rms_norm(mlstm_scan(q, k, v, i, f), None, eps).reshape(T, H * dv)
    return (o * w[pre + "norm"] * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------
def ff_dense(h, w: dict, pre: str):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def expert(h, w: dict, pre: str):
    return relu_squared(h @ w[pre + "up"].T) @ w[pre + "down"].T


def moe_route(h, w: dict, pre: str, top: int, margins=None):
    """(ids [T, top], weights [T, top]); margins (a list) receives, per token, the gap between the last chosen and the first rejected logit."""
    z = h @ w[pre + "router"].T + w[pre + "router.b"]
    order = np.argsort(-z, axis=-1, kind="stable")
    ids = order[:, :top]
    if margins is not None and top < z.shape[1]:
        zs = np.take_along_axis(z, order, -1)
        margins.extend((zs[:, top - 1] - zs[:, top]).tolist())
    zc = np.take_along_axis(z, ids, -1)
    e = np.exp(zc - zc.max(-1, keepdims=True))
    return ids, e / e.sum(-1, keepdims=True)


def ff_moe(h, w: dict, pre: str, mlp: dict, margins=None):
    ids, wts = moe_route(h, w, pre, int(mlp["router"]["top"]), margins)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(ids[t], wts[t]):
            out[t] += wt * expert(h[t:t + 1], w, f"{pre}e{e}.")[0]
    return out


# ---- model -------------------------------------------------------------------------------------------------------------
MIXERS = {"latent_attention": mixer_latent_attention, "mlstm": mixer_mlstm}


def forward(cfg: dict, w: dict, tokens, return_layers: bool = False, margins=None):
    """Logits [T, vocab] of the whole sequence (and, optionally, the residual stream after every layer [layers, T, E])."""
    eps = float(cfg["norm"]["eps"])
    x = embedding(cfg, w, tokens)
    trace = []
    for i, lc in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + MIXERS[lc["type"]](layer_norm(x, w[pre + "norm1"], eps), w, pre + "mix.", lc["mixer"], eps)
        mlp = lc.get("mlp")
        if mlp is not None:
            h = layer_norm(x, w[pre + "norm2"], eps)
            x = x + (ff_dense(h, w, pre + "mlp.") if mlp["kind"] == "dense" else ff_moe(h, w, pre + "mlp.", mlp, margins))
        trace.append(x.copy())
    logits = layer_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(trace)) if return_layers else logits


def load_dir(path: str):
    with open(f"{path}/config.json") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(f"{path}/model.safetensors")
