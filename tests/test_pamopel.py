"""Pamopel without a GPU: the plain evaluation against independent forms of its own equations, the configuration reader's
errors."""
import json
import math

import numpy as np
import pytest

import pamopel_cases as cases
import plain_pamopel as plain


def test_state_recurrence_equals_its_sum():
    rng = np.random.default_rng(3)
    T, H, G, N, dv = 23, 4, 2, 5, 3
    x, B, C = rng.normal(size=(T, H, dv)), rng.normal(size=(T, G, N)), rng.normal(size=(T, G, N))
    dt, lr, D = rng.uniform(0.01, 0.5, (T, H)), rng.normal(size=H), rng.normal(size=H)
    y = plain.selective_state(x, B, C, dt, lr, D)
    for h in range(H):
        g = h // 2
        for i in (0, 1, 9, T - 1):
            want = D[h] * x[i, h]
            for j in range(i + 1):
                want = want + math.exp(-math.exp(lr[h]) * dt[j + 1:i + 1, h].sum()) * dt[j, h] * (C[i, g] @ B[j, g]) * x[j, h]
            assert np.allclose(y[i, h], want)


def test_chunked_form_with_decays_per_token():
    """The algebra of the chunked kernels, every power the exponential of a difference of running sums."""
    rng = np.random.default_rng(4)
    T, L, N, dv, rate = 29, 8, 4, 6, -0.7
    x, B, C, dt = rng.normal(size=(T, dv)), rng.normal(size=(T, N)), rng.normal(size=(T, N)), rng.uniform(0, 1, T)
    want = plain.selective_state(x[:, None], B[:, None], C[:, None], dt[:, None], np.array([math.log(0.7)]), np.zeros(1))[:, 0]
    S, out = np.zeros((N, dv)), []
    for c in range(0, T, L):
        n = min(L, T - c)
        cum = np.cumsum(rate * dt[c:c + n])
        i = np.arange(n)
        w = np.where(i[:, None] >= i[None], np.exp(np.minimum(cum[:, None] - cum[None], 0)) * dt[None, c:c + n], 0)
        out.append((w * (C[c:c + n] @ B[c:c + n].T)) @ x[c:c + n] + np.exp(cum)[:, None] * (C[c:c + n] @ S))
        S = np.exp(cum[-1]) * S + ((dt[c:c + n] * np.exp(cum[-1] - cum))[:, None] * B[c:c + n]).T @ x[c:c + n]
    assert np.allclose(np.concatenate(out), want)


def test_convolution_reads_the_past_only():
    rng = np.random.default_rng(5)
    x, w, b = rng.normal(size=(9, 2)), rng.normal(size=(2, 4)), rng.normal(size=2)
    y = plain.causal_conv(x, w, b)
    assert np.allclose(y[0], b + w[:, 3] * x[0])
    assert np.allclose(y[5], b + w[:, 3] * x[5] + w[:, 2] * x[4] + w[:, 1] * x[3] + w[:, 0] * x[2])


def test_distance_buckets():
    of = lambda n: plain.distance_bucket(n, 12, 70)
    assert [of(n) for n in range(6)] == [0, 1, 2, 3, 4, 5] and of(6) == 6
    assert all(of(n) <= of(n + 1) for n in range(200))
    assert of(69) == 11 and of(70) == 11 and of(10 ** 6) == 11
    assert of(math.ceil(6 * (70 / 6) ** (1 / 6))) == 7 and of(math.ceil(6 * (70 / 6) ** (1 / 6)) - 1) == 6
    table = np.arange(24.0).reshape(12, 2)
    bias = plain.distance_bias(9, table, 70)
    assert bias.shape == (2, 9, 9) and bias[1, 8, 8] == table[0, 1] and bias[0, 8, 3] == table[5, 0]


def test_grouped_attention_of_one_key_head_is_shared():
    rng = np.random.default_rng(6)
    q, k, v = rng.normal(size=(7, 4, 5)), rng.normal(size=(7, 2, 5)), rng.normal(size=(7, 2, 3))
    out = plain.grouped_attention(q, k, v, 0.5, 0)
    for h in range(4):
        s = np.exp(q[6, h] @ k[:, h // 2].T * 0.5)
        assert np.allclose(out[6, h], s @ v[:, h // 2] / s.sum())
    assert np.allclose(out[0], v[0][[0, 0, 1, 1]])


def test_norm_over_parts_and_layer_norm():
    x = np.array([[3.0, 4.0, 0.0, 2.0]])
    assert np.allclose(plain.part_rms(x, 2, 0.0), [[3 / math.sqrt(12.5), 4 / math.sqrt(12.5), 0, math.sqrt(2)]])
    y = plain.layer_norm(x, np.array([1.0, 1.0, 1.0, 2.0]), 0.0)
    assert abs(y[0, :3].sum() + y[0, 3] / 2) < 1e-12 and abs((y[0, 0] ** 2 + y[0, 1] ** 2 + y[0, 2] ** 2 + y[0, 3] ** 2 / 4) / 4 - 1) < 1e-12


def test_embedding_pieces():
    assert plain.bigram_rows([4, 2, 4], 10, 3, 7) == [7, (40 + 6) % 7, (20 + 12) % 7]
    s = plain.sinusoid(3, 5)
    assert np.allclose(s[2], [math.sin(2), math.cos(2), math.sin(2 * 10000 ** -0.4), math.cos(2 * 10000 ** -0.4), math.sin(2 * 10000 ** -0.8)])


def test_a_borrowing_layer_uses_the_lender_s_keys():
    """Changing a lender's key weights changes what the borrower sees; the borrower has none of its own."""
    cfg = cases.CASES["borrowed"]
    t = cases.random_model(cfg, 2)
    assert "l1.mix.k" not in t and "l3.mix.v" not in t and "l1.mix.q" in t
    h = np.random.default_rng(1).normal(size=(6, cfg["width"]))
    w = plain.sub(t, "l1.mix.", np.float64)
    _, kv = plain.attention(h, plain.sub(t, "l0.mix.", np.float64), cfg["layers"][0]["mixer"], 1e-5, None)
    a, same = plain.attention(h, w, cfg["layers"][1]["mixer"], 1e-5, kv)
    b, _ = plain.attention(h, w, cfg["layers"][1]["mixer"], 1e-5, (kv[0][:, :, ::-1], kv[1]))
    assert same is kv and not np.allclose(a, b)


@pytest.fixture(scope="module")
def lib():
    from blok_b200 import build, lib
    build.build()
    return lib


def test_registry_names_the_design(lib):
    assert {"Pamopel", "Nomozen"} <= set(lib.architectures())


def test_configuration_errors_name_the_place(lib, tmp_path):
    """Refused while the configuration is read, before any device memory is taken."""
    def error(path, value=None, drop=False):
        cfg = json.loads(json.dumps(cases.CASES["borrowed"]))
        at = cfg
        for p in path[:-1]:
            at = at[p]
        if drop:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        with pytest.raises(lib.BlokError) as e:
            lib.Model.open(tmp_path)
        return str(e.value)
    for path, value, message in ((("layers", 0, "type"), "convolution", 'layer 0: unknown type "convolution"'),
                                 (("layers", 2, "mixer", "groups"), 3, "layer 2.mixer: groups does not divide the heads"),
                                 (("layers", 2, "mixer", "norm_groups"), 5, "layer 2.mixer: norm_groups does not divide the inner size"),
                                 (("layers", 2, "mixer", "conv"), 0, "layer 2.mixer: conv is not a positive integer"),
                                 (("layers", 0, "mixer", "kv_heads"), 3, "layer 0.mixer: kv_heads does not divide the heads"),
                                 (("layers", 1, "mixer", "kv_from"), 1, "layer 1.mixer: kv_from names no earlier attention layer"),
                                 (("layers", 3, "mixer", "kv_from"), 1, "layer 3.mixer: kv_from names no earlier attention layer"),
                                 (("layers", 3, "mixer", "kv_from"), 2, "layer 3.mixer: kv_from names no earlier attention layer"),
                                 (("layers", 1, "mixer", "dim"), 48, "layer 1.mixer: kv_from names no earlier attention layer"),
                                 (("layers", 1, "mixer", "bias_max"), 0, "layer 1.mixer: bias_max is not a distance"),
                                 (("layers", 1, "mlp", "kind"), "moe", 'layer 1: unknown feed-forward "moe"'),
                                 (("embedding", "bigram", "mul_cur"), -1, "a factor is negative"),
                                 (("layers",), [], "no layers")):
        assert message in error(path, value), path
    for path in (("residual_mult",), ("logit_scale",), ("embedding", "scale"), ("embedding", "bigram", "buckets"), ("norm", "eps"),
                 ("layers", 2, "mixer", "state"), ("layers", 0, "mixer", "scale"), ("layers", 0, "mlp", "ff")):
        assert path[-1] + " is missing" in error(path, drop=True), path
