"""Plain, slow evaluation of the Pamopel design in numpy (float64 unless told otherwise): one function per mechanism, token
by token or by the defining sums, no cache, no paging and no code of the product path.

A model here is (config, tensors): the parsed config.json and a dict name -> float array."""
import math

import numpy as np

from plain_nomozen import bf16_round, read_safetensors, rms, sigmoid, silu, sub, write_safetensors  # noqa: F401


# ---- embedding -------------------------------------------------------------------------------------------------------

def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """The row of the pair (previous token, token) at every position; the first position has a row of its own."""
    return [buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tokens[t]) * mul_cur) % buckets for t in range(len(tokens))]


def sinusoid(n, width):
    out = np.zeros((n, width))
    for i in range(width):
        rate = 10000.0 ** (-(i - i % 2) / width)
        out[:, i] = (np.cos if i % 2 else np.sin)(np.arange(n) * rate)
    return out


# ---- norms -----------------------------------------------------------------------------------------------------------

def layer_norm(x, w, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def part_rms(x, parts, eps):
    """Every one of `parts` equal pieces of the last axis over its own root mean square."""
    y = x.reshape(x.shape[:-1] + (parts, x.shape[-1] // parts))
    return rms(y, eps).reshape(x.shape)


# ---- selective state space -------------------------------------------------------------------------------------------

def causal_conv(x, w, b):
    """x [T, C], w [C, taps] with the current token's weight last."""
    T, taps = len(x), w.shape[1]
    out = np.zeros_like(x) + b
    for t in range(T):
        for j in range(taps):
            if t - j >= 0:
                out[t] += w[:, taps - 1 - j] * x[t - j]
    return out


def softplus(z):
    return np.maximum(z, 0) + np.log1p(np.exp(-np.abs(z)))


def selective_state(x, B, C, dt, log_rate, D):
    """x [T, H, v], B and C [T, G, N], dt [T, H]: S = exp(-exp(log_rate) dt) S + dt B x^T, y = S^T C + D x, one token after
    the other; head h uses group h // (H / G)."""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    S, y = np.zeros((H, N, dv), x.dtype), np.zeros_like(x)
    g = np.arange(H) // (H // G)
    for t in range(T):
        S = np.exp(-np.exp(log_rate) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t, g][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", S, C[t, g]) + D[:, None] * x[t]
    return y


def mamba2(h, w, m, eps):
    T, H, dv, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner].reshape(T, H, dv), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y = selective_state(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"]).reshape(T, inner)
    return (part_rms(y * silu(z), m["norm_groups"], eps) * w["norm"]) @ w["o"].T


# ---- softmax attention over grouped heads, a learned bias per distance -------------------------------------------------

def distance_bucket(n, rows, top):
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(top / half) * (rows - half)))


def distance_bias(T, table, top):
    """[H, T, T]: entry (h, i, j) is the bias of query i on key j (nothing behind the query is read)."""
    of = np.array([distance_bucket(n, len(table), top) for n in range(T)])
    d = np.maximum(np.arange(T)[:, None] - np.arange(T)[None], 0)
    return np.moveaxis(table[of[d]], -1, 0)


def grouped_attention(q, k, v, scale, bias):
    """q [T, H, d], k [T, G, d], v [T, G, dv], bias [H, T, T] or 0."""
    T, H, G = len(q), q.shape[1], k.shape[1]
    of = np.arange(H) // (H // G)
    s = np.einsum("ihd,jhd->hij", q, k[:, of]) * scale + bias
    s = np.where(np.tril(np.ones((T, T), bool))[None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return np.einsum("hij,jhd->ihd", p / p.sum(axis=-1, keepdims=True), v[:, of])


def attention(h, w, m, eps, kv):
    """kv: the keys and values of an earlier layer, or None; returns (output, keys and values)."""
    T, H, G, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w["q"].T, eps) * w["q.norm"]).reshape(T, H, d)
    if kv is None:
        kv = (rms(h @ w["k"].T, eps) * w["k.norm"]).reshape(T, G, d), (h @ w["v"].T).reshape(T, G, dv)
    o = grouped_attention(q, kv[0], kv[1], m["scale"], distance_bias(T, w["rel"], m["bias_max"]))
    o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T, kv


# ---- feed-forward and the whole model ----------------------------------------------------------------------------------

def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def forward(cfg, tensors, tokens, dtype=np.float64, layers=False):
    """Logits [T, vocab] of one sequence; with layers=True also the residual after every layer."""
    tokens = np.asarray(tokens)
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    top = {k: v.astype(dtype) for k, v in tensors.items() if k.split(".")[0] in ("embed", "bigram", "head", "final")}
    e = cfg["embedding"]
    b = e["bigram"]
    x = top["embed"][tokens] * e["scale"] + top["bigram"][bigram_rows(tokens, b["mul_prev"], b["mul_cur"], b["buckets"])]
    x = x + sinusoid(len(tokens), cfg["width"]).astype(dtype)
    trace, kept = [], {}
    for i, L in enumerate(cfg["layers"]):
        p = "l%d." % i
        w, wm, wf = sub(tensors, p, dtype), sub(tensors, p + "mix.", dtype), sub(tensors, p + "mlp.", dtype)
        h = layer_norm(x, w["norm1"], eps)
        if L["type"] == "mamba2":
            y = mamba2(h, wm, L["mixer"], eps)
        else:
            y, kept[i] = attention(h, wm, L["mixer"], eps, kept.get(L["mixer"].get("kv_from")))
        x = x + mult * layer_norm(y, w["norm1b"], eps)
        if L["mlp"] is not None:
            x = x + mult * layer_norm(gated_ff(layer_norm(x, w["norm2"], eps), wf), w["norm2b"], eps)
        trace.append(x)
    logits = layer_norm(x, top["final.norm"], eps) @ top["head"].T * cfg["logit_scale"]
    return (logits, np.stack(trace)) if layers else logits
