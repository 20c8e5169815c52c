"""Nomozen without a GPU: the plain evaluation against independent forms of its own equations, the configuration reader's
and the command line's errors."""
import json
import os
import subprocess

import numpy as np
import pytest

import nomozen_cases as cases
import plain_nomozen as plain

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_decayed_state_equals_its_sum():
    rng = np.random.default_rng(3)
    T, H, d, dv = 37, 3, 5, 7
    q, k, v = rng.normal(size=(T, H, d)), rng.normal(size=(T, H, d)), rng.normal(size=(T, H, dv))
    decay = [0.2, 0.9, 1.0]
    o = plain.decayed_state_attention(q, k, v, decay)
    for h in range(H):
        for i in (0, 1, 20, T - 1):
            want = sum(decay[h] ** (i - j) * (q[i, h] @ k[j, h]) * v[j, h] for j in range(i + 1))
            assert np.allclose(o[i, h], want)


def test_chunked_form_of_the_decayed_state():
    """The algebra of the chunked kernels: contributions of chunks, a scan, outputs inside a chunk plus the state before it."""
    rng = np.random.default_rng(4)
    T, C, d, dv, decay = 29, 8, 4, 6, 0.93
    q, k, v = rng.normal(size=(T, d)), rng.normal(size=(T, d)), rng.normal(size=(T, dv))
    want = plain.decayed_state_attention(q[:, None], k[:, None], v[:, None], [decay])[:, 0]
    S, out = np.zeros((d, dv)), []
    for c in range(0, T, C):
        n = min(C, T - c)
        qc, kc, vc = q[c:c + n], k[c:c + n], v[c:c + n]
        i = np.arange(n)
        w = np.where(i[:, None] >= i[None], decay ** np.maximum(i[:, None] - i[None], 0), 0)
        out.append((w * (qc @ kc.T)) @ vc + decay ** (i[:, None] + 1) * (qc @ S))
        S = decay ** n * S + (decay ** (n - 1 - i)[:, None] * kc).T @ vc
    assert np.allclose(np.concatenate(out), want)


def test_three_bf16_parts_hold_an_fp32_value():
    rng = np.random.default_rng(5)
    v = np.concatenate([rng.normal(size=4000), np.exp(rng.uniform(-30, 3, 4000))]).astype(np.float32)
    rest, total = v.copy(), np.zeros(v.size, np.float64)
    for _ in range(3):
        part = plain.bf16_round(rest)
        total += part
        rest = (rest - part).astype(np.float32)
    assert np.max(np.abs(total - v) / np.abs(v)) <= 2.0 ** -24


def test_rotation_is_relative():
    rng = np.random.default_rng(6)
    x, y = rng.normal(size=(1, 8)), rng.normal(size=(1, 8))
    dot = lambda p, r: float((plain.rotate_pairs(x, [p], 8, 1e4) @ plain.rotate_pairs(y, [r], 8, 1e4).T)[0, 0])
    assert abs(dot(7, 3) - dot(104, 100)) < 1e-9 and abs(dot(7, 3) - dot(7, 4)) > 1e-3
    part = plain.rotate_pairs(x, [5], 4, 1e4)
    assert np.array_equal(part[:, 4:], x[:, 4:]) and not np.allclose(part[:, :4], x[:, :4])


def test_looped_layers_run_in_a_row():
    assert plain.layer_order(cases.CASES["mixed"]) == [0, 1, 2, 1, 2, 1, 2, 3]
    assert plain.layer_order(cases.CASES["latent"]) == [0]


def test_one_stream_of_unit_mixing_is_the_plain_residual():
    x, y = np.ones((1, 2, 3)), np.full((2, 3), 5.0)
    assert np.array_equal(plain.mix_streams(x, y, np.eye(1), np.ones(1))[0], x[0] + y)
    two = np.stack([np.full((1, 3), 1.0), np.full((1, 3), 10.0)])  # mix is indexed [from, to]
    got = plain.mix_streams(two, np.zeros((1, 3)), np.array([[0.0, 1.0], [0.5, 0.0]]), np.zeros(2))
    assert np.array_equal(got[:, 0, 0], [5.0, 1.0])


@pytest.fixture(scope="module")
def lib():
    from blok_b200 import build, lib
    build.build()
    return lib


def test_registry_names_the_design(lib):
    assert "Nomozen" in lib.architectures()


def _open_error(lib, tmp_path, change, weights=True):
    cfg = json.loads(json.dumps(cases.CASES["mixed"]))
    change(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(lib.BlokError) as e:
        lib.Model.open(tmp_path)
    return str(e.value)


def test_configuration_errors_name_the_place(lib, tmp_path):
    """Refused while the configuration is read, before any device memory is taken."""
    def at(*path):
        def setter(cfg, value=None, drop=False):
            for p in path[:-1]:
                cfg = cfg[p]
            if drop:
                del cfg[path[-1]]
            else:
                cfg[path[-1]] = value
        return setter
    for path, value, message in ((("architecture",), "Unheard", 'architecture "Unheard" is not one of: '),
                                 (("layers", 0, "type"), "convolution", 'layer 0: unknown type "convolution"'),
                                 (("layers", 0, "mixer", "decay"), [0.5], "layer 0.mixer: decay has not one entry per head"),
                                 (("layers", 1, "mixer", "heads"), 0, "layer 1.mixer: heads is not a positive integer"),
                                 (("layers", 1, "mixer", "rot", "dims"), 7, "layer 1.mixer.rot: dims or base does not fit"),
                                 (("layers", 1, "mlp", "kind"), "dense", 'layer 1: unknown feed-forward "dense"'),
                                 (("loop", "stop"), 9, "the loop does not fit 4 layers"),
                                 (("streams",), 17, "17 residual streams (at most 16)")):
        assert message in _open_error(lib, tmp_path, lambda c: at(*path)(c, value)), path
    for path in (("width",), ("norm", "eps"), ("layers", 2, "mixer", "vdim"), ("layers", 0, "mlp", "router", "top"), ("layers", 3, "mixer", "scale")):
        assert path[-1] + " is missing" in _open_error(lib, tmp_path, lambda c: at(*path)(c, drop=True)), path
    (tmp_path / "config.json").write_text("{\"architecture\": \"Nomozen\",}")
    with pytest.raises(lib.BlokError, match="config.json: expected a field name"):
        lib.Model.open(tmp_path)


def test_command_line_errors(lib):
    exe = os.path.join(ROOT, "blok_b200", "blok-kimi-exec")
    run = lambda *a: subprocess.run([exe, *a], capture_output=True, text=True, timeout=60)
    p = run("--model", "/nonexistent", "--prompt-tokens", "1", "--tokens", "1")
    assert p.returncode == 1 and "cannot open /nonexistent/config.json" in p.stderr
    p = run("--model", "x", "--dtype", "half", "--prompt-tokens", "1", "--tokens", "1")
    assert p.returncode == 1 and "unknown dtype: half" in p.stderr
    trace = os.path.join(ROOT, "bin", "trace_run")
    p = subprocess.run([trace, "--model", "/nonexistent", "--dtype", "bfloat16", "--out", "/tmp", "--max-tokens", "8"], input="", capture_output=True,
                       text=True, timeout=600)
    assert p.returncode == 1 and "cannot open /nonexistent/config.json" in p.stderr
