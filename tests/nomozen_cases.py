"""Small Nomozen configurations of the tests (sizes that need padding, sizes that do not, one of everything)."""
import json
import os

import plain_nomozen as plain


def linear(kind, heads, dim, vdim, decay, mlp=None):
    return {"type": kind, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, q_rank, base=10000.0, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
                      "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5}}


def experts(n, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def config(width, vocab, streams, layers, loop=None, eps=1e-5):
    c = {"architecture": "Nomozen", "width": width, "vocab": vocab, "streams": streams, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # each mixer alone, no feed-forward, one stream; sizes that are multiples of nothing
    "retention": config(72, 101, 1, [linear("retention", 3, 20, 24, [0.5, 0.97, 0.999])]),
    "lightning": config(104, 77, 1, [linear("lightning", 5, 36, 28, [0.3, 0.8, 0.95, 0.99, 1.0])], eps=1e-2),
    "latent": config(88, 97, 1, [latent(5, 24, 12, 40, 56, 28)]),
    # experts behind the cheapest mixer; one expert per token, and three
    "one_expert": config(64, 96, 2, [linear("retention", 1, 16, 16, [0.9], experts(7, 1, 48))]),
    "three_experts": config(96, 120, 2, [linear("retention", 2, 16, 32, [0.9, 0.99], experts(11, 3, 40))]),
    # everything: unequal layers, a loop in the middle, five streams
    "mixed": config(160, 203, 5, [linear("lightning", 4, 48, 16, [0.6, 0.9, 0.99, 0.999], experts(6, 2, 72)),
                                  latent(3, 40, 8, 24, 72, 44, base=500.0, mlp=experts(9, 3, 24)),
                                  linear("retention", 2, 32, 80, [0.98, 0.9995]),
                                  latent(18, 32, 32, 16, 136, 64, scale=0.2, mlp=experts(4, 1, 32))], loop=(1, 3, 3)),
    # no padding anywhere, sizes of the wide kernels: more than 16 heads, K a multiple of 256, a rank over 256
    "aligned": config(256, 512, 4, [latent(32, 64, 64, 64, 288, 256, mlp=experts(8, 2, 256)),
                                    linear("retention", 4, 128, 128, [0.9, 0.97, 0.99, 0.999], experts(8, 2, 256))]),
    # the row size of the tcgen05 attention core
    "core": config(64, 96, 2, [latent(24, 64, 64, 128, 512, 64), latent(70, 32, 64, 16, 512, 32)]),
    # latents too wide for the tensor-core kernel, heads too wide for the prompt kernel
    "wide": config(64, 80, 3, [latent(2, 264, 8, 16, 40, 32), latent(2, 16, 40, 16, 520, 32),
                               linear("lightning", 1, 240, 64, [0.97])]),
}


GAIN = {"mixed": 0.7}  # smaller matrices keep the eight layer runs from amplifying rounding


def write(directory, name, seed=1, edit=None):
    """The case's folder (config.json, model.safetensors); returns (config, tensors)."""
    cfg = CASES[name]
    tensors = plain.random_model(cfg, seed, GAIN.get(name, 1.0))
    if edit:
        edit(cfg, tensors)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    plain.write_safetensors(os.path.join(directory, "model.safetensors"), tensors)
    return cfg, tensors
