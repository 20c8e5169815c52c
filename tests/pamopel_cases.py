"""Small Pamopel configurations of the tests (sizes that need padding, sizes that do not, one of everything) and their random
weights."""
import json
import math
import os

import numpy as np

import plain_pamopel as plain


def state(heads, vdim, n, groups=1, taps=4, norm_groups=1, ff=None):
    return {"type": "mamba2", "mlp": ff and {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "vdim": vdim, "state": n, "groups": groups, "conv": taps, "norm_groups": norm_groups}}


def attn(heads, kv_heads, dim, vdim, bias_max=40, buckets=8, scale=None, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "scale": scale or 1.3 * dim ** -0.5, "_buckets": buckets}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": ff and {"kind": "dense", "ff": ff}}


def config(width, vocab, layers, buckets=101, mul_prev=13, mul_cur=5, scale=3.0, mult=0.6, logit_scale=1.5, eps=1e-5):
    return {"architecture": "Pamopel", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_scale": logit_scale, "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


CASES = {
    # each mixer alone, no feed-forward; sizes that are multiples of nothing
    "state": config(72, 101, [state(6, 20, 24, groups=3, taps=3, norm_groups=4)]),
    "state_plain": config(40, 64, [state(1, 16, 16, taps=1)], mult=1.0, logit_scale=1.0, scale=1.0),
    "attention": config(88, 97, [attn(6, 2, 24, 40, bias_max=70, buckets=12)], eps=1e-3),
    "one_head": config(66, 83, [attn(1, 1, 20, 12, bias_max=5, buckets=2)], buckets=7),
    # keys and values borrowed twice, by layers with feed-forward of their own; a state-space layer with one
    "borrowed": config(96, 120, [attn(8, 1, 40, 24, ff=72), attn(8, 1, 40, 24, bias_max=90, buckets=6, scale=0.3, kv_from=0, ff=40),
                                 state(4, 36, 40, groups=2, taps=5, norm_groups=3, ff=88), attn(8, 1, 40, 24, kv_from=0)]),
    # everything, unequal layers of each kind
    "mixed": config(160, 203, [state(4, 24, 48, groups=4, taps=2, norm_groups=2), attn(12, 3, 72, 56, bias_max=33, buckets=16, ff=104),
                               state(10, 16, 20, groups=5, taps=6, norm_groups=8, ff=56), attn(10, 5, 32, 64, bias_max=300, buckets=20),
                               attn(12, 3, 72, 56, bias_max=64, buckets=4, kv_from=1, ff=33), attn(20, 1, 16, 16)], buckets=1000, mul_prev=1000003),
    # no padding anywhere, sizes of the wide kernels: K a multiple of 256, heads of 64 and 128, more than 16 heads to a key head
    "aligned": config(256, 512, [state(8, 64, 128, groups=1, norm_groups=1), attn(16, 4, 128, 128, bias_max=128, buckets=32, ff=512),
                                 attn(24, 1, 64, 64, bias_max=128, buckets=32, ff=256)]),
    # heads too wide for the tcgen05 kernel (values), for every tensor-core kernel, states of 256 rows
    "wide": config(64, 80, [attn(2, 1, 256, 144), attn(2, 2, 320, 272), state(2, 80, 240, groups=2)]),
}
GAIN = {}


def random_model(cfg, seed, gain=1.0):
    """Seeded weights (exact bfloat16 values) of the shapes the configuration asks for."""
    rng = np.random.default_rng(seed)
    W, V, t = cfg["width"], cfg["vocab"], {}
    mat = lambda name, r, c, g=1.0: t.__setitem__(name, plain.bf16_round(rng.normal(size=(r, c)).astype(np.float32) * (g * gain / math.sqrt(c))))
    vec = lambda name, n, mean=1.0, dev=0.2: t.__setitem__(name, plain.bf16_round((mean + dev * rng.normal(size=n)).astype(np.float32)))
    mat("embed", V, W, math.sqrt(W) / cfg["embedding"]["scale"])
    mat("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, W, math.sqrt(W))
    for i, L in enumerate(cfg["layers"]):
        p, m = "l%d." % i, L["mixer"]
        vec(p + "norm1", W)
        vec(p + "norm1b", W)
        if L["type"] == "mamba2":
            inner, bc = m["heads"] * m["vdim"], m["groups"] * m["state"]
            mat(p + "mix.in", 2 * inner + 2 * bc + m["heads"], W)
            mat(p + "mix.conv", inner + 2 * bc, m["conv"], 1.5)
            vec(p + "mix.conv.b", inner + 2 * bc, 0.1, 0.2)
            vec(p + "mix.dt_bias", m["heads"], -2.0, 1.5)
            vec(p + "mix.A_log", m["heads"], 0.3, 0.8)
            vec(p + "mix.D", m["heads"], 0.8, 0.5)
            vec(p + "mix.norm", inner)
            mat(p + "mix.o", W, inner)
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * d, W)
            vec(p + "mix.q.norm", H * d)
            if m.get("kv_from") is None:
                mat(p + "mix.k", G * d, W)
                vec(p + "mix.k.norm", G * d)
                mat(p + "mix.v", G * dv, W)
            t[p + "mix.rel"] = plain.bf16_round(rng.normal(size=(m["_buckets"], H)).astype(np.float32) * 1.5)
            mat(p + "mix.g", H, W, 1.5)
            mat(p + "mix.o", W, H * dv)
        if L["mlp"] is not None:
            vec(p + "norm2", W)
            vec(p + "norm2b", W)
            ff = L["mlp"]["ff"]
            mat(p + "mlp.gate", ff, W, 1.4)
            mat(p + "mlp.up", ff, W)
            mat(p + "mlp.down", W, ff)
    vec("final.norm", W)
    mat("head", V, W, 2.0)
    return t


def write(directory, name, seed=1, edit=None):
    """The case's folder (config.json, model.safetensors); returns (config, tensors)."""
    cfg = json.loads(json.dumps(CASES[name]))
    tensors = random_model(cfg, seed, GAIN.get(name, 1.0))
    if edit:
        edit(cfg, tensors)
    stored = json.loads(json.dumps(cfg))
    for L in stored["layers"]:
        L["mixer"].pop("_buckets", None)  # the table's shape says it
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(stored, f)
    plain.write_safetensors(os.path.join(directory, "model.safetensors"), tensors)
    return cfg, tensors
