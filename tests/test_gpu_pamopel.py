"""Pamopel on the GPU against the plain evaluation (plain_pamopel.py): every mechanism through its own entry point, whole
models in fp32 (tight) and bf16, prompts against portions against single tokens, batches against each sequence alone,
slots and pages that are used again, generation through the scheduler."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import pamopel_cases as cases
import plain_pamopel as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# Root mean square of a row's error against the logits' spread; bf16: the median row and the largest.
TIGHT, LOOSE, WORST = 1e-4, 3e-2, 0.1


def bf16(a, device):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).to(device).bfloat16()


def f32(a, device):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).to(device)


def i32(a, device):
    return torch.tensor(a, dtype=torch.int32, device=device)


def f64(t):
    return t.float().cpu().numpy().astype(np.float64)


def row_errors(got, want):
    d = got - want
    return np.sqrt((d * d).mean(axis=-1)) / want.std()


def assert_rows(got, want, dtype, what=""):
    e = row_errors(got, want)
    if dtype == "float32":
        assert e.max() < TIGHT, "%s: %.2e at %d" % (what, e.max(), int(e.argmax()))
    else:
        assert np.median(e) < LOOSE and e.max() < WORST, "%s: median %.2e, %.2e at %d" % (what, np.median(e), e.max(), int(e.argmax()))


def tokens_of(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def feed(model, slot, tokens, sizes):
    """The sequence in portions of the given sizes (cycled); the logits at every position."""
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[k % len(sizes)], len(tokens) - at)
        out.append(model.extend(slot, tokens[at:at + n], range(n)))
        at, k = at + n, k + 1
    return np.concatenate(out)


# ---- mechanisms alone --------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("T,R,K", [(1, 16, 32), (65, 36, 72), (129, 260, 136), (300, 1000, 512)])
def test_gated_product(cuda, T, R, K):
    from blok_b200 import lib
    g = torch.Generator(device=cuda).manual_seed(T + R)
    x = torch.randn((T, K), generator=g, device=cuda).bfloat16()
    w = (torch.randn((2 * R, K), generator=g, device=cuda) * K ** -0.5).bfloat16()
    y = x.double() @ w.double().T
    want = torch.nn.functional.silu(y[:, :R]) * y[:, R:]
    got = lib.gemm_swiglu(x, w)
    assert float((got.double() - want).abs().max() / want.abs().max()) < 5e-3


@pytest.mark.parametrize("width,true", [(32, 20), (96, 96), (640, 637), (1536, 1530), (4096, 4096), (7168, 7150), (9216, 9200)])
def test_residual_norm(cuda, width, true):
    from blok_b200 import lib
    rng = np.random.default_rng(width)
    T, eps, mult = 3, 1e-2, 0.35
    pad = lambda a: np.pad(a, [(0, 0)] * (a.ndim - 1) + [(0, width - true)]).astype(np.float32)
    x, y = pad(rng.normal(size=(T, true)) + 40), pad(rng.normal(size=(T, true)) * 0.1 - 3)  # means far from zero
    post, w = pad(rng.normal(size=true)), pad(rng.normal(size=true))
    dx = f32(x, cuda)
    got = f64(lib.residual_norm(dx, f32(y, cuda), f32(post, cuda), mult, f32(w, cuda), eps, true))
    x64, y64 = x[:, :true].astype(np.float64), y[:, :true].astype(np.float64)
    x1 = x64 + mult * plain.layer_norm(y64, post[:true], eps)
    assert np.abs(f64(dx)[:, :true] - x1).max() < 2e-5 and np.abs(f64(dx)[:, true:]).max(initial=0) == 0
    want = plain.layer_norm(x1, w[:true], eps)
    assert np.abs(got[:, :true] - want).max() < 1e-4 and np.abs(got[:, true:]).max(initial=0) == 0
    half = f64(lib.residual_norm(dx, None, None, mult, f32(w, cuda), eps, true, f32=False))
    assert np.abs(half[:, :true] - want).max() < 5e-3 * np.abs(want).max()
    lib.residual_norm(dx, f32(y, cuda), None, mult, f32(w, cuda), eps, true)  # a plain sum
    assert np.abs(f64(dx)[:, :true] - (x1 + mult * y64)).max() < 3e-5


def test_token_embedding(cuda):
    """A prompt in two portions and decoding of several sequences: the previous token is carried per slot, the first token has
    the last row; large factors need 64 bits; far positions keep their angles."""
    from blok_b200 import lib
    rng = np.random.default_rng(3)
    vocab, width, true, buckets, mp, mc, scale = 50, 32, 30, 37, 4000000007, 3000000019, 2.5
    e, b = (plain.bf16_round(np.pad(rng.normal(size=(n, true)), [(0, 0), (0, width - true)]).astype(np.float32)) for n in (vocab, buckets + 1))
    turns = torch.tensor([10000.0 ** (-2 * i / true) / (2 * np.pi) for i in range(width // 2)], dtype=torch.float64, device=cuda)
    tok = rng.integers(0, vocab, 12)
    want = e[tok].astype(np.float64) * scale + b[plain.bigram_rows(tok, mp, mc, buckets)]
    want[:, :true] += plain.sinusoid(12, true)
    last = torch.full((4,), 49, dtype=torch.int32, device=cuda)  # what former sequences left

    def run(ids, slots, pos, chunk, keep=True):
        return f64(lib.token_embedding(i32(ids, cuda), last, i32(slots, cuda), i32(pos, cuda), chunk, keep, bf16(e, cuda), bf16(b, cuda), buckets, mp, mc,
                                       scale, turns, true))
    got = [run(tok[:5].tolist(), [2] * 5, range(5), True), run(tok[5:7].tolist(), [2] * 2, [5, 6], True)]
    assert np.abs(run([int(tok[0])], [1], [0], False) - want[:1]).max() < 1e-5  # another sequence starts beside it
    for t in range(7, 12):
        both = run([int(tok[t]), int(tok[t - 6])], [2, 1], [t, t - 6], False)
        got.append(both[:1])
        assert np.abs(both[1:] - want[t - 6:t - 5]).max() < 1e-5
    assert np.abs(np.concatenate(got) - want).max() < 1e-5
    assert last.tolist() == [49, int(tok[5]), int(tok[11]), 49]
    far = run([1], [0], [1000003], False, keep=False)[0, :true] - run([1], [0], [1], False, keep=False)[0, :true]
    angle = 10000.0 ** (-(np.arange(true) // 2 * 2) / true)
    exact = np.where(np.arange(true) % 2, np.cos(1000003 * angle) - np.cos(angle), np.sin(1000003 * angle) - np.sin(angle))
    assert np.abs(far - exact).max() < 2e-5


def state_weights(rng, heads, channels, taps):
    return (rng.normal(size=(taps, channels)).astype(np.float32), rng.normal(size=channels).astype(np.float32) * 0.3,
            rng.normal(size=heads).astype(np.float32) - 1, -np.exp(rng.normal(size=heads)).astype(np.float32))


@pytest.mark.parametrize("heads,channels,taps", [(3, 48, 4), (40, 80, 1), (33, 32, 2), (5, 144, 7)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_state_inputs(cuda, heads, channels, taps, dtype):
    """Portions shorter and longer than the convolution and the chunk, single tokens in between, a slot that was in use."""
    from blok_b200 import lib
    rng = np.random.default_rng(heads + taps)
    sizes = [1, 2, 70, 1, 1, 3, 64, 2, 1, 129]
    T, first, dt_at = sum(sizes), 16, 16 + channels
    proj = plain.bf16_round(rng.normal(size=(T, dt_at + (heads + 15) // 16 * 16)).astype(np.float32))
    cw, cb, db, rate = state_weights(rng, heads, channels, taps)
    x = torch.from_numpy(proj).to(cuda).to(dtype)
    ring = torch.full((3, taps, channels), 9.0, device=cuda, dtype=dtype)
    dev = [f32(a, cuda) for a in (cw, cb, db, rate)]
    at, outs = 0, []
    want = plain.silu(plain.causal_conv(proj[:, first:dt_at].astype(np.float64), cw.T.astype(np.float64), cb))
    dt = plain.softplus(proj[:, dt_at:dt_at + heads].astype(np.float64) + db)
    for n in sizes:
        out, tok = lib.state_inputs(x[at:at + n].contiguous(), first, dt_at, heads, *dev, ring, i32([1] * n, cuda), i32(range(at, at + n), cuda), n > 1)
        outs.append(f64(out))
        tok = tok.cpu().numpy().astype(np.float64)
        lg = dt[at:at + n] * rate
        assert np.abs(tok[:, :, 0].T - dt[at:at + n]).max() < 1e-5 and np.abs(tok[:, :, 1].T - lg).max() < 1e-5 * np.abs(lg).max()
        for c in range(0, n, 64):
            cum = np.cumsum(tok[:, c:c + 64, 1], axis=1)
            assert np.abs(tok[:, c:c + 64, 2] + tok[:, c:c + 64, 3] - cum).max() < 1e-7 * max(1.0, np.abs(cum).max())
        at += n
    got = np.concatenate(outs)
    assert np.abs(got - want).max() < (1e-5 if dtype == torch.float32 else 6e-3) * np.abs(want).max()
    assert float((ring[[0, 2]] - 9.0).abs().max()) == 0, "other slots are untouched"


def test_state_inputs_of_several_sequences(cuda):
    from blok_b200 import lib
    rng = np.random.default_rng(1)
    heads, channels, taps, B = 4, 32, 4, 5
    cw, cb, db, rate = state_weights(rng, heads, channels, taps)
    dev = [f32(a, cuda) for a in (cw, cb, db, rate)]
    ring = torch.full((6, taps, channels), 5.0, device=cuda)
    slots, lens = [4, 0, 5, 2, 1], [0, 1, 2, 3, 9]
    seqs = [rng.normal(size=(n + 1, channels + 16)).astype(np.float32) for n in lens]
    for s, n, a in zip(slots, lens, seqs):
        if n:
            lib.state_inputs(f32(a[:n], cuda), 0, channels, heads, *dev, ring, i32([s] * n, cuda), i32(range(n), cuda), True)
    out, _ = lib.state_inputs(f32(np.stack([a[-1] for a in seqs]), cuda), 0, channels, heads, *dev, ring, i32(slots, cuda), i32(lens, cuda), False)
    for i, a in enumerate(seqs):
        want = plain.silu(plain.causal_conv(a[:, :channels].astype(np.float64), cw.T, cb))[-1]
        assert np.abs(f64(out)[i] - want).max() < 1e-5, i


def token_rows(dt, rate):
    """[heads, T, 4] as the kernels take them: chunks of 64 start at row 0."""
    T, H = dt.shape
    lg = (dt * rate).astype(np.float32)
    out = np.zeros((H, T, 4), np.float32)
    out[:, :, 0], out[:, :, 1] = dt.T, lg.T
    for c in range(0, T, 64):
        cum = np.cumsum(lg[c:c + 64].astype(np.float64), axis=0)
        hi = cum.astype(np.float32)
        out[:, c:c + 64, 2], out[:, c:c + 64, 3] = hi.T, (cum - hi).T
    return out


@pytest.mark.parametrize("H,G,N,dv", [(1, 1, 16, 16), (6, 3, 48, 80), (4, 1, 128, 64), (4, 4, 240, 32), (8, 2, 32, 144)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_selective_state_portions_and_steps(cuda, H, G, N, dv, dtype):
    """Portions around the 64-token chunk, then single tokens, on one carried state; steps from almost 0 to decays of e^-60."""
    from blok_b200 import lib
    rng = np.random.default_rng(H * N + dv)
    sizes = [65, 2, 64, 1, 130, 9, 63, 8, 1, 1]
    T, ld = sum(sizes), H * dv + 2 * G * N
    a = plain.bf16_round(rng.normal(size=(T, ld)).astype(np.float32))
    dt = np.exp(rng.uniform(-7, 1.5, (T, H))).astype(np.float32)
    dt[rng.random((T, H)) < 0.02] = 30.0
    log_rate, D = rng.normal(size=H) * 0.7, rng.normal(size=H).astype(np.float32)
    rate = -np.exp(log_rate).astype(np.float32)
    x, B, C = a[:, :H * dv].reshape(T, H, dv), a[:, H * dv:H * dv + G * N].reshape(T, G, N), a[:, H * dv + G * N:].reshape(T, G, N)
    want = plain.selective_state(*(v.astype(np.float64) for v in (x, B, C, dt)), np.log(-rate.astype(np.float64)), D.astype(np.float64)).reshape(T, H * dv)
    state = torch.full((3, H, N, dv), 7.0, device=cuda)  # what a former sequence left behind
    t, skip = torch.from_numpy(a).to(cuda).to(dtype), f32(D, cuda)
    at, got = 0, []
    for n in sizes:
        part, tok = t[at:at + n].contiguous(), f32(token_rows(dt[at:at + n], rate), cuda)
        where = dict(slot_of=i32([2], cuda), pos=i32([at], cuda)) if n == 1 else dict(slot=2, first_pos=at)
        got.append(lib.selective_state(part, H, G, N, dv, tok, skip, state, **where))
        at += n
    got = f64(torch.cat(got))
    assert np.max(np.abs(got - want)) / np.abs(want).max() < 5e-6
    assert float((state[:2] - 7.0).abs().max()) == 0, "other slots are untouched"


def test_selective_state_keeps_a_far_token(cuda):
    """One token written far back and read by one query: lost if a chunk's state is dropped or decays by a step too many."""
    from blok_b200 import lib
    H, N, dv, T, far = 2, 32, 32, 400, 67
    ask = [68, 127, 128, 129, 191, 192, 399]
    a = np.zeros((T, H * dv + 2 * N), np.float32)
    a[far, :H * dv] = plain.bf16_round(np.random.default_rng(1).normal(size=H * dv).astype(np.float32))
    a[far, H * dv + 3] = 1
    a[ask, H * dv + N + 3] = 1
    dt, rate = np.random.default_rng(2).uniform(0.0, 0.02, (T, H)).astype(np.float32), np.array([-1.0, -3.0], np.float32)
    got = f64(lib.selective_state(bf16(a, cuda), H, 1, N, dv, f32(token_rows(dt, rate), cuda), torch.zeros(H, device=cuda), torch.zeros((1, H, N, dv), device=cuda)))
    for i in ask:
        for h in range(H):
            want = dt[far, h] * np.exp((dt[far + 1:i + 1, h].astype(np.float64) * rate[h]).sum()) * a[far, h * dv:(h + 1) * dv]
            assert np.abs(got[i, h * dv:(h + 1) * dv] - want).max() <= 1e-5 * np.abs(want).max(), (i, h)
    assert np.abs(got[:far]).max() == 0


@pytest.mark.parametrize("heads,vdim,true,parts", [(3, 16, 16, 1), (6, 32, 20, 4), (7, 48, 48, 7), (1, 16, 9, 3), (64, 64, 64, 2), (5, 16, 15, 25)])
def test_gate_then_norm(cuda, heads, vdim, true, parts):
    """Parts that cut heads in the middle, with and without padding; the gate changes what the norm sees."""
    from blok_b200 import lib
    rng = np.random.default_rng(heads + parts)
    T, eps = 4, 1e-3
    o, g, w = rng.normal(size=(T, heads, vdim)) * 0.1, rng.normal(size=(T, heads, vdim)) * 2, rng.normal(size=(heads, vdim))
    for a in (o, g, w):
        a[..., true:] = 0
    o32, g32, w32 = (a.reshape(a.shape[:-2] + (-1,)).astype(np.float32) for a in (o, g, w))
    cut = lambda a: a.reshape(a.shape[:-1] + (heads, vdim))[..., :true].reshape(a.shape[:-1] + (-1,)).astype(np.float64)
    for dtype, bar in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        dg = torch.from_numpy(g32).to(cuda).to(dtype)
        got = f64(lib.gate_then_norm(f32(o32, cuda), dg, heads, vdim, true, parts, eps, f32(w32, cuda)))
        want = plain.part_rms(cut(o32) * plain.silu(cut(f64(dg))), parts, eps) * cut(w32)
        assert np.abs(cut(got) - want).max() < bar * np.abs(want).max()
        assert np.abs(got.reshape(T, heads, vdim)[..., true:]).max(initial=0) == 0


def paged(rows, page, slots, device, seed=0):
    """`rows` [n, row] laid out in shuffled pages: (pool, table whose last slot holds them); other pages hold large values."""
    n = len(rows)
    pages = (n + page - 1) // page
    order = np.random.default_rng(seed).permutation(pages + 3)[:pages]
    pool = torch.full((pages + 3, page, rows.shape[1]), 50.0, dtype=rows.dtype, device=device)
    for j in range(pages):
        part = rows[j * page:(j + 1) * page]
        pool[int(order[j]), :len(part)] = part
    table = torch.zeros((slots, pages), dtype=torch.int32)
    table[slots - 1] = torch.from_numpy(order.astype(np.int32))
    return pool, table.to(device)


def test_grouped_append(cuda):
    from blok_b200 import lib
    rng = np.random.default_rng(4)
    H, G, d, true, dv, T, page, eps = 6, 2, 64, 40, 48, 37, 32, 1e-2
    ld = H * d + G * (d + dv) + 16
    a = np.zeros((T, ld), np.float32)
    cut = lambda x, n: x.reshape(T, n, d)[:, :, :true]
    for lo, n in ((0, H), (H * d, G)):
        a[:, lo:lo + n * d].reshape(T, n, d)[:, :, :true] = rng.normal(size=(T, n, true)) * 0.2
    a[:, (H + G) * d:] = rng.normal(size=(T, ld - (H + G) * d))
    qn, kn = np.zeros(H * d, np.float32), np.zeros(G * d, np.float32)
    qn.reshape(H, d)[:, :true], kn.reshape(G, d)[:, :true] = rng.normal(size=(H, true)), rng.normal(size=(G, true))
    for dtype, bar in ((torch.float32, 1e-5), (torch.bfloat16, 5e-3)):
        x = torch.from_numpy(a).to(cuda).to(dtype)
        src = f64(x)
        row = G * (d + dv)
        pool, table = paged(torch.zeros((70, row), device=cuda, dtype=dtype), page, 2, cuda)
        first = 30  # crosses a page
        lib.grouped_append(x, H, G, d, true, dv, f32(qn, cuda), f32(kn, cuda), eps, table, i32([1] * T, cuda), i32(range(first, first + T), cuda), pool)
        norm = lambda lo, n, w: plain.rms(cut(src[:, lo:lo + n * d], n).reshape(T, -1), eps).reshape(T, n, true) * w.reshape(n, d)[None, :, :true]
        q, k = norm(0, H, qn), norm(H * d, G, kn)
        got = f64(x)
        assert np.abs(cut(got[:, :H * d], H) - q).max() < bar * np.abs(q).max() and np.array_equal(got[:, H * d:], src[:, H * d:])
        order = table[1].tolist()
        flat = np.concatenate([f64(pool[p]) for p in order])[:70]
        assert np.abs(cut(flat[first:first + T, :G * d], G) - k).max() < bar * np.abs(k).max()
        assert np.array_equal(flat[first:first + T, G * d:], src[:, (H + G) * d:(H + G) * d + G * dv])
        assert np.abs(flat[:first]).max() == 0 and np.abs(flat[first + T:]).max() == 0
        before = pool.clone()
        lib.grouped_append(x, H, G, d, true, dv, f32(qn, cuda), None, eps, table, None, None, None)  # a borrowing layer: queries only
        assert torch.equal(before, pool) and not np.array_equal(f64(x)[:, :H * d], got[:, :H * d])


def bias_table(rng, H, n, jumps=()):
    """By distance; at the given distances one entry stands out, so that a distance that is one off shows."""
    b = rng.normal(size=(H, n)).astype(np.float32)
    for j in {j for j in jumps if j < n}:
        b[:, j] += 9 * (-1) ** j
    return b


def attend_plain(q, k, v, pos, scale, bias, gate):
    """q [T, H, d] at positions pos, k [n, G, d], v [n, G, dv], bias [H, len] or None, gate [T, H] or None."""
    T, H = q.shape[:2]
    of = np.arange(H) // (H // k.shape[1])
    out = np.zeros((T, H, v.shape[2]))
    for i, p in enumerate(pos):
        s = np.einsum("hd,jhd->hj", q[i], k[:p + 1, of]) * scale
        if bias is not None:
            s = s + bias[:, np.minimum(p - np.arange(p + 1), bias.shape[1] - 1)]
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = np.einsum("hj,jhv->hv", w / w.sum(axis=1, keepdims=True), v[:p + 1, of])
    return out if gate is None else out * plain.sigmoid(gate)[:, :, None]


def grouped_inputs(rng, n, H, G, d, dv, pos):
    """Rows and queries with one key per query standing out: its own, the first, a middle one, at the edges of tiles of 64."""
    rows = rng.normal(size=(n, G * (d + dv))).astype(np.float32)
    q = rng.normal(size=(len(pos), H, d)).astype(np.float32) * 0.3
    k = rows[:, :G * d].reshape(n, G, d)
    of = np.arange(H) // (H // G)
    for i, p in enumerate(pos):
        star = [p, 0, p // 2, max(0, p - 64), p // 64 * 64, max(0, p // 64 * 64 - 1), max(0, p - 1)][i % 7]
        q[i] += k[star, of] * 2
    return plain.bf16_round(rows), plain.bf16_round(q)


@pytest.mark.parametrize("H,G,d,dv,blen,dtype", [
    (1, 1, 32, 16, 1, torch.bfloat16), (6, 2, 64, 80, 65, torch.bfloat16), (14, 1, 96, 112, 210, torch.bfloat16), (32, 8, 128, 128, 0, torch.bfloat16),
    (40, 2, 64, 64, 129, torch.bfloat16), (3, 3, 160, 208, 500, torch.bfloat16), (17, 1, 256, 256, 33, torch.bfloat16), (4, 2, 320, 272, 40, torch.bfloat16),
    (6, 3, 96, 48, 70, torch.float32), (5, 1, 32, 16, 0, torch.float32)])
@pytest.mark.parametrize("page", [32, 64])
def test_grouped_attend(cuda, H, G, d, dv, blen, dtype, page):
    """Positions at the edges of tiles, pages, context splits and the bias table's end."""
    from blok_b200 import lib
    rng = np.random.default_rng(H + d + dv)
    n = 1000
    pos = [0, 1, 62, 63, 64, 65, 127, 128, 129, 500, 640, 998, 999]
    rows, q = grouped_inputs(rng, n, H, G, d, dv, pos)
    bias = bias_table(rng, H, blen, {0, 1, blen // 2, blen - 1}) if blen else None
    gate = plain.bf16_round(rng.normal(size=(len(pos), H)).astype(np.float32) * 2) if H != 32 else None
    pool, table = paged(torch.from_numpy(rows).to(cuda).to(dtype), page, 3, cuda)
    got = f64(lib.grouped_attend(torch.from_numpy(q).to(cuda).to(dtype), pool, table, i32([2] * len(pos), cuda), i32(pos, cuda), G, dv, 0.25, n,
                                 None if bias is None else f32(bias, cuda), None if gate is None else torch.from_numpy(gate).to(cuda).to(dtype)))
    k, v = rows[:, :G * d].reshape(n, G, d).astype(np.float64), rows[:, G * d:].reshape(n, G, dv).astype(np.float64)
    want = attend_plain(q.astype(np.float64), k, v, pos, 0.25, bias, gate)
    bar = 2e-5 if dtype == torch.float32 else 5e-3  # bf16: the output's own rounding
    for i, p in enumerate(pos):
        assert np.max(np.abs(got[i] - want[i])) < bar * np.abs(want[i]).max(), p


@pytest.mark.parametrize("H,G,d,dv,blen", [(1, 1, 32, 16, 1), (6, 2, 64, 80, 65), (10, 2, 96, 112, 210), (4, 2, 128, 128, 0), (3, 3, 160, 64, 500),
                                           (2, 1, 256, 112, 33), (5, 5, 224, 48, 1000)])
@pytest.mark.parametrize("T,n,page", [(33, 33, 32), (200, 200, 64), (64, 321, 32), (129, 257, 96), (40, 1000, 64)])
def test_grouped_prompt(cuda, H, G, d, dv, blen, T, n, page):
    from blok_b200 import lib
    rng = np.random.default_rng(H + d + T)
    pos = list(range(n - T, n))
    rows, q = grouped_inputs(rng, n, H, G, d, dv, pos)
    bias = bias_table(rng, H, blen, {0, 1, blen // 2, blen - 1}) if blen else None
    gate = plain.bf16_round(rng.normal(size=(T, H)).astype(np.float32) * 2) if blen != 65 else None
    scale = 0.25 if blen != 33 else -0.25  # with a bias the scale may have any sign
    pool, table = paged(bf16(rows, cuda), page, 2, cuda)
    got = f64(lib.grouped_prompt(bf16(q, cuda), pool, table, 1, n, G, dv, scale, None if bias is None else f32(bias, cuda),
                                 None if gate is None else bf16(gate, cuda)))
    k, v = rows[:, :G * d].reshape(n, G, d).astype(np.float64), rows[:, G * d:].reshape(n, G, dv).astype(np.float64)
    want = attend_plain(q.astype(np.float64), k, v, pos, scale, bias, gate)
    err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max(axis=(1, 2))
    assert err.max() < 6e-3, (int(err.argmax()), err.max())


def test_bias_moves_attention_by_one_distance(cuda):
    """Equal keys: the biases alone decide.  One distance stands out; the value found there is that key's, at every edge."""
    from blok_b200 import lib
    n, d, dv = 400, 32, 16
    rows = np.zeros((n, d + dv), np.float32)
    rows[:, d:] = plain.bf16_round(np.random.default_rng(3).normal(size=(n, dv)).astype(np.float32))
    pool, table = paged(bf16(rows, cuda), 32, 1, cuda)
    for dist in (0, 1, 31, 32, 63, 64, 65, 127, 191, 192, 254):
        bias = np.full((1, 256), -40.0, np.float32)
        bias[0, dist] = 0.0
        for T in (400, 100):
            got = f64(lib.grouped_prompt(torch.zeros((T, 1, d), dtype=torch.bfloat16, device=cuda), pool, table, 0, n, 1, dv, 1.0, f32(bias, cuda)))[:, 0]
            i = np.arange(max(dist, n - T), n)
            assert np.abs(got[i - (n - T)] - rows[i - dist, d:]).max() < 1e-2, (dist, T)
        i = np.array([p for p in (dist, dist + 1, 63, 64, 255, 256, 399) if p >= dist])
        got = f64(lib.grouped_attend(torch.zeros((len(i), 1, d), dtype=torch.bfloat16, device=cuda), pool, table, i32([0] * len(i), cuda), i32(i, cuda), 1, dv,
                                     1.0, n, f32(bias, cuda)))[:, 0]
        assert np.abs(got - rows[i - dist, d:]).max() < 1e-2, dist


# ---- whole models ------------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            d = tmp_path_factory.mktemp(name)
            made[name] = (str(d),) + cases.write(str(d), name, seed=len(name))
        return made[name]
    return get


@pytest.mark.parametrize("name", sorted(cases.CASES))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_model_matches_plain(cuda, folder, name, dtype):
    """Every layer's residual and every logit of a prompt, then the same tokens in portions and one by one."""
    from blok_b200 import lib
    d, cfg, tensors = folder(name)
    T = 150
    tok = tokens_of(cfg, T, 5)
    want, layers = plain.forward(cfg, tensors, tok, layers=True)
    model = lib.Model.open(d, dtype=dtype, max_batch=2, max_ctx=160, prefill_chunk=160, kv_page_rows=32)
    trace = model.trace_layers(T)
    got = model.extend(0, tok, range(T))
    run = f64(trace)
    for i in range(len(layers)):
        assert_rows(run[i], layers[i], dtype, "after layer %d" % i)
    model.trace_layers(0)
    assert_rows(got, want, dtype, "prompt")
    model.release_slot(0)
    for sizes in ([2], [3, 33, 1, 64, 7], [100, 1]):
        assert_rows(feed(model, 1, tok, sizes), want, dtype, "portions of %s" % sizes)
        model.release_slot(1)
    assert_rows(feed(model, 0, tok, [1]), want, dtype, "token by token")
    model.check()
    model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "aligned"])
def test_prompts_longer_than_a_chunk_and_long_decoding(cuda, folder, name, dtype):
    from blok_b200 import lib
    d, cfg, tensors = folder(name)
    tok = tokens_of(cfg, 420, 6)
    model = lib.Model.open(d, dtype=dtype, max_ctx=420, prefill_chunk=96)
    got = np.concatenate([model.extend(0, tok[:230], range(230)), feed(model, 0, tok[230:], [1])])
    assert_rows(got, plain.forward(cfg, tensors, tok), dtype)
    model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["attention", "state"])
def test_far_token_decides(cuda, tmp_path, case, dtype):
    """A far token answers the last query (sharp queries, or few large steps and slow decays): exchanging it must move the last logits as the plain
    evaluation says, from a prompt and from decoding alike."""
    from blok_b200 import lib

    def sharpen(cfg, t):
        if case == "attention":
            t["l0.mix.q.norm"] = plain.bf16_round(t["l0.mix.q.norm"] * 8)
        else:
            t["l0.mix.A_log"] = plain.bf16_round(t["l0.mix.A_log"] - 5)
            t["l0.mix.dt_bias"] = plain.bf16_round(t["l0.mix.dt_bias"] - 6)
            t["l0.mix.in"][-cfg["layers"][0]["mixer"]["heads"]:] *= 4
    cfg, tensors = cases.write(str(tmp_path), case, seed=8, edit=sharpen)
    T = 210
    tok = np.random.default_rng(11).integers(0, cfg["vocab"], T)
    base, most = plain.forward(cfg, tensors, tok)[-1], (0.0, None, None)
    for far in range(0, 60, 3):
        other = tok.copy()
        other[far] = (tok[far] + 1) % cfg["vocab"]
        moved = plain.forward(cfg, tensors, other)[-1] - base
        if moved.std() > most[0]:
            most = (moved.std(), other, moved)
    assert most[0] > 0.03 * base.std(), "a far token matters"
    model = lib.Model.open(str(tmp_path), dtype=dtype, max_batch=3, max_ctx=256, kv_page_rows=32)
    for sizes in ([T], [T - 1, 1], [64, 1], [2]):
        got = []
        for x in (tok, most[1]):
            got.append(feed(model, 1, x.tolist(), sizes)[-1])
            model.release_slot(1)
        bar = 1e-3 if dtype == "float32" else 0.3
        assert np.sqrt(((got[1] - got[0] - most[2]) ** 2).mean()) < bar * most[0], sizes
    model.close()


@pytest.mark.parametrize("name", ["mixed", "aligned"])
def test_steps_of_unequal_sequences_equal_each_alone(cuda, folder, name):
    """Twelve sequences of different lengths step together (greedy ids, several batch sizes, slots in any order)."""
    from blok_b200 import lib
    d, cfg, tensors = folder(name)
    model = lib.Model.open(d, dtype="float32", max_batch=12, max_ctx=96, prefill_chunk=64, kv_page_rows=32)
    seqs = [tokens_of(cfg, 1 + 7 * i % 50, 20 + i) for i in range(12)]
    for s, tok in enumerate(seqs):
        model.extend(s, tok)
    torch.cuda.synchronize()  # the steps run on a stream of their own, from graphs where a batch size comes again
    side = torch.cuda.Stream()
    with torch.cuda.stream(side):
        for step, slots in enumerate(([3, 0, 11, 7, 5, 1, 2, 4, 6, 8, 9, 10], [2, 9, 4], [7], [11, 10, 9, 8, 7, 6, 5, 4, 3, 2, 1, 0], [9, 2, 4], [4, 2, 9])):
            ids = [(31 * step + 5 * s) % cfg["vocab"] for s in slots]
            nxt = model.step_slots(slots, i32(ids, cuda))
            for s, t in zip(slots, ids):
                seqs[s] = seqs[s] + [t]
            side.synchronize()
            for s, got in list(zip(slots, nxt.tolist()))[:4]:
                logits = plain.forward(cfg, tensors, seqs[s])[-1]
                assert logits[got] >= logits.max() - 1e-3 * logits.std(), (step, s)
    model.close()


def test_bf16_batches_agree_with_single_sequences(cuda, folder):
    """The products of a step change their kernels with the batch size: the same sequence alone, in a batch of 5 and of 40."""
    from blok_b200 import lib
    d, cfg, tensors = folder("aligned")
    model = lib.Model.open(d, max_batch=41, max_ctx=64, prefill_chunk=64, kv_page_rows=32)
    tok = tokens_of(cfg, 20, 3)
    want = plain.forward(cfg, tensors, tok + [5])[-1]
    for batch in (1, 5, 40):
        for s in range(batch):
            model.extend(s, tok if s == batch - 1 else tokens_of(cfg, 3 + s, 50 + s))
        slots = list(range(batch))
        nxt = model.step_slots(slots, torch.full((batch,), 5, dtype=torch.int32, device=cuda))
        got = int(nxt[-1])
        assert want[got] > want.max() - 0.05 * want.std(), batch
        again = model.extend(batch - 1, [7], [0])[0]
        exp = plain.forward(cfg, tensors, tok + [5, 7])[-1]
        assert_rows(again[None], exp[None], "bfloat16", batch)
        for s in range(batch):
            model.release_slot(s)
    model.check()
    model.close()


def test_slots_and_pages_are_used_again(cuda, folder):
    from blok_b200 import lib
    d, cfg, tensors = folder("mixed")
    model = lib.Model.open(d, dtype="float32", max_batch=2, max_ctx=128, prefill_chunk=64, kv_page_rows=32, kv_pages=5)
    long, short = tokens_of(cfg, 120, 1), tokens_of(cfg, 30, 2)
    want_short = plain.forward(cfg, tensors, short)
    for _ in range(3):
        model.extend(0, long)
        with pytest.raises(lib.BlokError, match="free pages"):
            model.extend(1, long[:40])
        assert model.slot_length(1) == 0 and model.free_pages == 1
        assert row_errors(model.extend(1, short, range(30)), want_short).max() < TIGHT
        model.release_slot(0)
        model.release_slot(1)
        assert model.free_pages == 5
        assert row_errors(feed(model, 0, short, [11, 1]), want_short).max() < TIGHT
        model.release_slot(0)
        assert row_errors(feed(model, 1, short, [1]), want_short).max() < TIGHT
        model.release_slot(1)
    with pytest.raises(lib.BlokError, match="exceed max_ctx"):
        model.extend(0, long + long)
    with pytest.raises(lib.BlokError, match="outside the vocabulary"):
        model.extend(0, [cfg["vocab"]])
    model.close()


def greedy(cfg, tensors, prompt, n):
    """(tokens, smallest gap between the best and the second logit, in spreads)"""
    out, gap = list(prompt), np.inf
    for _ in range(n):
        logits = plain.forward(cfg, tensors, out)[-1]
        top = np.sort(logits)[-2:]
        gap = min(gap, (top[1] - top[0]) / logits.std())
        out.append(int(np.argmax(logits)))
    return out[len(prompt):], gap


def test_generation_through_the_scheduler(cuda, folder):
    """generate, generate_many (more requests than slots, a pool that holds only some) and the command line."""
    from blok_b200 import lib
    d, cfg, tensors = folder("mixed")
    prompts = [tokens_of(cfg, n, 40 + n) for n in (3, 40, 1, 17, 66)]
    want = [greedy(cfg, tensors, p, 12) for p in prompts]
    model = lib.Model.open(d, dtype="float32", max_batch=3, max_ctx=96, prefill_chunk=32, kv_page_rows=32, kv_pages=6)
    one = model.generate(prompts[1], 12)
    many = model.generate_many(prompts, 12)
    model.close()
    sure = [i for i, w in enumerate(want) if w[1] > 1e-3]
    assert len(sure) >= 3
    for i in sure:
        assert many[i] == want[i][0], i
    assert one == many[1]
    exe = os.path.join(ROOT, "blok_b200", "blok-kimi-exec")
    p = subprocess.run([exe, "--model", d, "--dtype", "float32", "--prompt-tokens", ",".join(map(str, prompts[1])), "--tokens", "12"],
                       capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert json.loads(p.stdout)["token_ids"] == one


def test_replay_of_a_trace(cuda, folder, tmp_path):
    """bin/trace_run: interleaved sequences, portions, ends; the files hold the wanted rows."""
    d, cfg, tensors = folder("mixed")
    a, b = tokens_of(cfg, 70, 1), tokens_of(cfg, 33, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[50:51], "want": [0]}, {"id": "b", "tokens": a[:2], "want": [1]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[51:], "want": [18]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [32]}], "end": ["b"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "120"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done %d" % i for i in range(5)]
    la, lb = plain.forward(cfg, tensors, a), plain.forward(cfg, tensors, b + a[:2])
    for step, rows in ((0, la[[0, 49]]), (2, np.stack([la[50], lb[34]])), (3, la[69:70]), (4, lb[32:33])):
        got = np.fromfile(tmp_path / ("%d.f32" % step), np.float32).reshape(-1, cfg["vocab"])
        assert got.shape == rows.shape and row_errors(got, rows).max() < TIGHT, step
    assert not (tmp_path / "1.f32").exists()


def test_missing_and_misshapen_tensors_are_named(cuda, tmp_path):
    from blok_b200 import lib
    for edit, message in ((lambda c, t: t.pop("l0.mix.conv.b"), "missing tensor l0.mix.conv.b"),
                          (lambda c, t: t.pop("l1.mix.rel"), "tensor l1.mix.rel is missing"),
                          (lambda c, t: t.__setitem__("l0.mix.in", t["l0.mix.in"][:-1]), "tensor l0.mix.in has another type, shape or size"),
                          (lambda c, t: t.__setitem__("bigram", t["bigram"][:-1]), "tensor bigram has another type, shape or size"),
                          (lambda c, t: c["layers"][1]["mixer"].__setitem__("bias_max", 8), "l1.mix.rel: 16 buckets up to a distance of 8")):
        cases.write(str(tmp_path), "mixed", edit=edit)
        with pytest.raises(lib.BlokError, match=message):
            lib.Model.open(str(tmp_path))
