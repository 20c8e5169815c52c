"""Plain, slow evaluation of the Nomozen design in numpy (float64 unless told otherwise): one function per mechanism,
token by token or by the defining sums, no cache, no paging and no code of the product path.

A model here is (config, tensors): the parsed config.json and a dict name -> float array (int array for the expert
tables)."""
import json
import math
import struct

import numpy as np


# ---- files ---------------------------------------------------------------------------------------------------------

def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 value (ties to even), returned as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    r = ((u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)).astype(np.uint32)
    return r.view(np.float32).reshape(np.shape(a))


def read_safetensors(path):
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        lo, hi = t["data_offsets"]
        data = raw[8 + n + lo:8 + n + hi]
        if t["dtype"] == "BF16":
            a = (np.frombuffer(data, np.uint16).astype(np.uint32) << 16).view(np.float32)
        elif t["dtype"] == "F32":
            a = np.frombuffer(data, np.float32)
        else:
            a = np.frombuffer(data, np.int32)
        out[name] = a.reshape(t["shape"])
    return out


def write_safetensors(path, tensors):
    head, blobs, at = {}, [], 0
    for name, a in tensors.items():
        if a.dtype.kind == "f":
            data = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
            dt = "BF16"
        else:
            data, dt = np.ascontiguousarray(a, np.int32).tobytes(), "I32"
        head[name] = {"dtype": dt, "shape": list(a.shape), "data_offsets": [at, at + len(data)]}
        blobs.append(data)
        at += len(data)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


# ---- elementwise pieces ----------------------------------------------------------------------------------------------

def silu(z):
    return z / (1 + np.exp(-z))


def sigmoid(z):
    return 1 / (1 + np.exp(-z))


def rms(x, eps):
    """x over the root of its mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(x, alpha, w, b):
    return np.tanh(alpha * x) * w + b


def rotate_pairs(x, pos, dims, base):
    """x [T, ..., n]: dimensions (2i, 2i + 1), i < dims / 2, turned by pos * base^(-2i / dims)."""
    y = x.copy()
    for i in range(dims // 2):
        a = np.asarray(pos, x.dtype) * x.dtype.type(base ** (-2.0 * i / dims))
        a = a.reshape([-1] + [1] * (x.ndim - 2))
        c, s = np.cos(a), np.sin(a)
        y[..., 2 * i] = x[..., 2 * i] * c - x[..., 2 * i + 1] * s
        y[..., 2 * i + 1] = x[..., 2 * i + 1] * c + x[..., 2 * i] * s
    return y


# ---- token mixers: h [T, width] of one sequence from its first token on ------------------------------------------------

def decayed_state_attention(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv]: S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, one token after the other."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype)
    o = np.zeros((T, H, v.shape[2]), q.dtype)
    dec = np.asarray(decay, q.dtype)[:, None, None]
    for t in range(T):
        S = dec * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def retention(h, w, m, eps):
    T, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d)
    k = (h @ w["k"].T).reshape(T, H, d) * d ** -0.5
    v = (h @ w["v"].T).reshape(T, H, dv)
    o = rms(decayed_state_attention(q, k, v, m["decay"]), eps)
    return (o.reshape(T, H * dv) * silu(h @ w["g"].T)) @ w["o"].T


def lightning(h, w, m, eps):
    T, H, d, dv = len(h), m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).reshape(T, H, d)
    k = silu(h @ w["k"].T).reshape(T, H, d)
    v = silu(h @ w["v"].T).reshape(T, H, dv)
    o = decayed_state_attention(q, k, v, m["decay"]).reshape(T, H * dv)
    return (rms(o, eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def latent_attention(h, w, m, eps):
    T, H, d, r, dv, c = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = ((rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).reshape(T, H, d + r)
    ckr = h @ w["dkv"].T
    lat = rms(ckr[:, :c], eps) * w["dkv.norm"]
    kr = rotate_pairs(ckr[:, c:], pos, m["rot"]["dims"], m["rot"]["base"])
    qr = rotate_pairs(q[:, :, d:], pos, m["rot"]["dims"], m["rot"]["base"])
    k = (lat @ w["uk"].T).reshape(T, H, d)
    v = (lat @ w["uv"].T).reshape(T, H, dv)
    s = (np.einsum("ihd,jhd->hij", q[:, :, :d], k) + np.einsum("ihr,jr->hij", qr, kr)) * m["scale"]
    s = np.where(np.tril(np.ones((T, T), bool))[None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    p = p / p.sum(axis=-1, keepdims=True)
    return np.einsum("hij,jhd->ihd", p, v).reshape(T, H * dv) @ w["o"].T


MIXERS = {"retention": retention, "lightning": lightning, "latent_attention": latent_attention}


# ---- feed-forward ----------------------------------------------------------------------------------------------------

def table_experts(h, tokens, w, m):
    """Each token's experts come from the table's row of its id; squared-ReLU experts, equal weights 1 / top."""
    y = np.zeros_like(h)
    top = m["router"]["top"]
    for t, tok in enumerate(tokens):
        for e in w["table"][tok]:
            up = np.maximum(w["e%d.up" % e] @ h[t], 0)
            y[t] += (w["e%d.down" % e] @ (up * up)) / top
    return y


# ---- residual streams and the whole model ------------------------------------------------------------------------------

def mix_streams(x, y, mix, out):
    """x [s, T, width]: x'_t = sum_s mix[s, t] x_s + out[t] y, all from the old x."""
    return np.einsum("st,snw->tnw", mix, x) + out[:, None, None] * y[None]


def layer_order(cfg):
    """Indices of the layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def sub(tensors, prefix, dtype):
    return {k[len(prefix):]: (v.astype(dtype) if v.dtype.kind == "f" else v) for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, dtype=np.float64, layers=False):
    """Logits [T, vocab] of one sequence; with layers=True also the summed streams after every layer run."""
    tokens = np.asarray(tokens)
    eps = cfg["norm"]["eps"]
    norm = lambda x, w, name: dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])
    top = {k: v.astype(dtype) for k, v in tensors.items() if k.split(".")[0] in ("embed", "head", "final")}
    x = np.repeat(top["embed"][tokens][None], cfg["streams"], axis=0)
    trace, cached = [], {}
    for i in layer_order(cfg):
        L = cfg["layers"][i]
        if i not in cached:
            p = "l%d." % i
            cached[i] = (sub(tensors, p, dtype), sub(tensors, p + "mix.", dtype), sub(tensors, p + "mlp.", dtype))
        w, wm, wf = cached[i]
        u = np.einsum("s,snw->nw", w["hc1.in"], x)
        y = MIXERS[L["type"]](norm(u, w, "norm1"), wm, L["mixer"], eps)
        x = mix_streams(x, y, w["hc1.mix"], w["hc1.out"])
        if L["mlp"] is not None:
            u = np.einsum("s,snw->nw", w["hc2.in"], x)
            y = table_experts(norm(u, w, "norm2"), tokens, wf, L["mlp"])
            x = mix_streams(x, y, w["hc2.mix"], w["hc2.out"])
        trace.append(x.sum(axis=0))
    logits = norm(x.sum(axis=0), top, "final.norm") @ top["head"].T
    return (logits, np.stack(trace)) if layers else logits


# ---- random small models -----------------------------------------------------------------------------------------------

def random_model(cfg, seed, gain=1.0):
    """Seeded weights (exact bfloat16 values) of the shapes the configuration asks for."""
    rng = np.random.default_rng(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    t = {}
    mat = lambda name, r, c, g=1.0: t.__setitem__(name, bf16_round(rng.normal(size=(r, c)).astype(np.float32) * (g * gain / math.sqrt(c))))
    vec = lambda name, n, mean=1.0, dev=0.2: t.__setitem__(name, bf16_round((mean + dev * rng.normal(size=n)).astype(np.float32)))

    def norm(name):
        vec(name, W)
        vec(name + ".b", W, 0.0, 0.1)
        t[name + ".alpha"] = bf16_round(np.float32(0.7 + 0.4 * rng.random()).reshape(()))
    t["embed"] = bf16_round(rng.normal(size=(V, W)).astype(np.float32))
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        norm(p + "norm1")
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "latent_attention":
            r, c, qr = m["rot_dim"], m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", qr, W)
            vec(p + "mix.dq.norm", qr)
            mat(p + "mix.uq", H * (d + r), qr, 1.5)
            mat(p + "mix.dkv", c + r, W)
            vec(p + "mix.dkv.norm", c)
            mat(p + "mix.uk", H * d, c, 1.5)
            mat(p + "mix.uv", H * dv, c)
            mat(p + "mix.o", W, H * dv, 1.5)
        else:
            for n, rows in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                mat(p + "mix." + n, rows, W)
            mat(p + "mix.o", W, H * dv, 1.5)
            if L["type"] == "lightning":
                vec(p + "mix.norm", H * dv)
        hcs = ["hc1"]
        if L["mlp"] is not None:
            norm(p + "norm2")
            E, k, ff = L["mlp"]["router"]["experts"], L["mlp"]["router"]["top"], L["mlp"]["expert"]["ff"]
            for e in range(E):
                mat(p + "mlp.e%d.up" % e, ff, W, 1.4)
                mat(p + "mlp.e%d.down" % e, W, ff)
            t[p + "mlp.table"] = np.stack([rng.permutation(E)[:k] for _ in range(V)]).astype(np.int32)
            hcs.append("hc2")
        for hc in hcs:
            vec(p + hc + ".in", S, 1.0 / S, 0.3 / S)
            vec(p + hc + ".out", S, 1.0, 0.3)
            t[p + hc + ".mix"] = bf16_round((0.7 * np.eye(S) + 0.3 / S * rng.normal(size=(S, S))).astype(np.float32))
    norm("final.norm")
    mat("head", V, W, 2.0)
    return t
