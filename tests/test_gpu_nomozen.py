"""Nomozen on the GPU against the plain evaluation (plain_nomozen.py): every mechanism through its own entry point, whole
models in fp32 (tight) and bf16, prompts against portions against single tokens, batches against each sequence alone,
slots and pages that are used again, generation through the scheduler."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import nomozen_cases as cases
import plain_nomozen as plain

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# Root mean square of a row's error against the logits' spread.  fp32: the largest row.  bf16: the median row; single rows
# may lie higher (a first token's retention output has the sign of one dot product), a wrong row lies near 1.
TIGHT, LOOSE, WORST = 2e-4, 8e-2, 0.3


def bf16(a, device):
    return torch.from_numpy(np.ascontiguousarray(a, np.float32)).to(device).bfloat16()


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

@pytest.mark.parametrize("T,R,K", [(1, 16, 32), (9, 48, 96), (129, 260, 72), (300, 1000, 520), (128, 128, 64), (1000, 4352, 1024)])
def test_gemm(cuda, T, R, K):
    from blok_b200 import lib
    g = torch.Generator(device=cuda).manual_seed(T + R)
    x = torch.randn((T, K), generator=g, device=cuda).bfloat16()
    w = torch.randn((R, K), generator=g, device=cuda).bfloat16()
    want = x.double() @ w.double().T
    got = lib.gemm_bf16(x, w)
    assert float((got.double() - want).abs().max() / want.abs().max()) < 2e-6
    sq = torch.relu(want) ** 2
    got = lib.gemm_bf16(x, w, relu2=True, f32=False)
    assert float((got.double() - sq).abs().max() / sq.abs().max()) < 5e-3


def linear_inputs(rng, T, H, d, dv, extra=16):
    return plain.bf16_round(rng.normal(size=(T, 2 * H * d + H * dv + extra)).astype(np.float32))


def split_qkv(a, H, d, dv):
    T = len(a)
    a = a.astype(np.float64)
    return a[:, :H * d].reshape(T, H, d), a[:, H * d:2 * H * d].reshape(T, H, d), a[:, 2 * H * d:2 * H * d + H * dv].reshape(T, H, dv)


@pytest.mark.parametrize("H,d,dv", [(1, 16, 16), (3, 64, 80), (2, 128, 128), (2, 240, 48), (4, 32, 144)])
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
def test_linear_attention_portions_and_steps(cuda, H, d, dv, dtype):
    """Portions around the 64-token chunk, then single tokens, on one carried state; decays from 0 to 1."""
    from blok_b200 import lib
    rng = np.random.default_rng(H * d + dv)
    sizes = [65, 2, 64, 1, 130, 9, 63, 8, 1, 1]
    T = sum(sizes)
    a = linear_inputs(rng, T, H, d, dv)
    q, k, v = split_qkv(a, H, d, dv)
    decay = ([0.0, 0.9, 0.999, 1.0] if H > 1 else [0.97])[:H]
    scale = d ** -0.5
    want = plain.decayed_state_attention(q, k * scale, v, decay).reshape(T, H * dv)
    state = torch.full((3, H, d, dv), 7.0, device=cuda)  # what a former sequence left behind
    x = torch.from_numpy(a).to(cuda).to(dtype)
    at, got = 0, []
    for n in sizes:
        part = x[at:at + n].contiguous()
        if n == 1:
            slot_of, pos = (torch.tensor([i], dtype=torch.int32, device=cuda) for i in (2, at))
            got.append(lib.linear_attention(part, H, d, dv, decay, scale, False, state, slot_of=slot_of, pos=pos))
        else:
            got.append(lib.linear_attention(part, H, d, dv, decay, scale, False, state, slot=2, first_pos=at))
        at += n
    got = f64(torch.cat(got))
    assert np.max(np.abs(got - want)) / np.abs(want).max() < 5e-6
    assert float((state[:2] - 7.0).abs().max()) == 0, "other slots are untouched"
    S = np.zeros((H, d, dv))
    for t in range(T):
        S = np.asarray(decay)[:, None, None] * S + scale * k[t][:, :, None] * v[t][:, None, :]
    assert np.max(np.abs(f64(state[2]) - S)) / np.abs(S).max() < 5e-6


def test_linear_attention_keeps_a_far_token(cuda):
    """One key far back, found again by one query: lost if a chunk's state is dropped or decays by a step too many."""
    from blok_b200 import lib
    H, d, dv, T = 2, 32, 32, 400
    a = np.zeros((T, 2 * H * d + H * dv), np.float32)
    far, ask = 67, [68, 127, 128, 129, 191, 192, 399]
    a[far, H * d:2 * H * d] = np.tile(np.eye(d)[3], H)
    a[far, 2 * H * d:] = plain.bf16_round(np.random.default_rng(1).normal(size=H * dv).astype(np.float32))
    a[ask, :H * d] = np.tile(np.eye(d)[3], H)
    decay = [0.98, 0.5]
    q, k, v = split_qkv(a, H, d, dv)
    want = plain.decayed_state_attention(q, k, v, decay).reshape(T, H * dv)
    got = f64(lib.linear_attention(bf16(a, cuda), H, d, dv, decay, 1.0, False, torch.zeros((1, H, d, dv), device=cuda)))
    for t in ask:
        assert np.max(np.abs(got[t] - want[t])) <= 1e-5 * np.abs(want[t, :dv]).max(), t
    assert np.abs(got[:far]).max() == 0


def test_linear_attention_step_of_several_sequences(cuda):
    from blok_b200 import lib
    H, d, dv, B = 3, 48, 32, 7
    rng = np.random.default_rng(9)
    state = torch.zeros((9, H, d, dv), device=cuda)
    slots = [4, 0, 8, 2, 5, 1, 7]
    prompts = [plain.bf16_round(rng.normal(size=(3 + 11 * i, 2 * H * d + H * dv)).astype(np.float32)) for i in range(B)]
    last = plain.bf16_round(rng.normal(size=(B, 2 * H * d + H * dv)).astype(np.float32))
    for s, p in zip(slots, prompts):
        lib.linear_attention(bf16(p, cuda), H, d, dv, [0.9, 0.99, 1.0], 1.0, True, state, slot=s)
    got = f64(lib.linear_attention(bf16(last, cuda), H, d, dv, [0.9, 0.99, 1.0], 1.0, True, state,
                                   slot_of=torch.tensor(slots, dtype=torch.int32, device=cuda),
                                   pos=torch.tensor([len(p) for p in prompts], dtype=torch.int32, device=cuda)))
    for i, p in enumerate(prompts):
        a = plain.bf16_round(plain.silu(np.concatenate([p, last[i:i + 1]]).astype(np.float64)).astype(np.float32))
        want = plain.decayed_state_attention(*split_qkv(a, H, d, dv), [0.9, 0.99, 1.0])[-1].ravel()
        assert np.max(np.abs(got[i] - want)) / np.abs(want).max() < 2e-3, i  # SiLU may round to the neighbouring bf16 value


@pytest.mark.parametrize("per_head,sigmoid,weight", [(True, False, False), (False, True, True)])
def test_gated_norm(cuda, per_head, sigmoid, weight):
    from blok_b200 import lib
    rng = np.random.default_rng(2)
    T, H, dv, true, eps = 5, 11, 48, 44, 1e-2
    o, g, w = rng.normal(size=(T, H, dv)) * 0.05, rng.normal(size=(T, H * dv)) * 3, rng.normal(size=H * dv)
    o[:, :, true:] = 0
    o32, g32, w32 = (np.asarray(a, np.float32) for a in (o.reshape(T, -1), g, w))
    got = f64(lib.gated_norm(torch.from_numpy(o32).to(cuda), torch.from_numpy(g32).to(cuda), H, dv, true, per_head, eps, sigmoid,
                             torch.from_numpy(w32).to(cuda) if weight else None))
    x = o32.astype(np.float64).reshape(T, H, dv)[:, :, :true]
    n = plain.rms(x, eps) if per_head else plain.rms(x.reshape(T, -1), eps).reshape(T, H, true)
    want = np.zeros((T, H, dv))
    want[:, :, :true] = n
    want = want.reshape(T, -1) * (w32 if weight else 1.0) * (plain.sigmoid(g32) if sigmoid else plain.silu(g32.astype(np.float64)))
    assert np.max(np.abs(got - want)) < 1e-5 * np.abs(want).max()


def paged(rows, page, table_rows, device, seed=0):
    """`rows` [n, row] laid out in shuffled pages: (pool, one-slot table); other pages hold large values."""
    n = len(rows)
    pages = (n + page - 1) // page
    order = np.random.default_rng(seed).permutation(pages + 3)[:pages]
    pool = torch.full((pages + 3, page, rows.shape[1]), 50.0, dtype=rows.dtype, device=device)
    for j in range(pages):
        part = rows[j * page:(j + 1) * page]
        pool[int(order[j]), :len(part)] = part
    table = torch.zeros((table_rows, pages), dtype=torch.int32)
    table[table_rows - 1] = torch.from_numpy(order.astype(np.int32))
    return pool, table.to(device)


def attend_plain(q, rows, rank, scale, pos):
    out = np.zeros((len(pos), q.shape[1], rank))
    for i, p in enumerate(pos):
        s = q[i] @ rows[:p + 1].T * scale
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = (w / w.sum(axis=1, keepdims=True)) @ rows[:p + 1, :rank]
    return out


@pytest.mark.parametrize("H,rank,rot,dtype", [(1, 32, 32, torch.bfloat16), (5, 96, 32, torch.bfloat16), (16, 224, 64, torch.bfloat16),
                                              (40, 512, 64, torch.bfloat16), (64, 512, 64, torch.bfloat16), (17, 160, 32, torch.bfloat16), (3, 544, 32, torch.bfloat16),
                                              (6, 96, 32, torch.float32)])
@pytest.mark.parametrize("core", ["own choice", "mma"])
def test_latent_attend(cuda, monkeypatch, H, rank, rot, dtype, core):
    """Positions at the edges of tiles, pages and context splits; one key per query stands out somewhere (the first, a far
    one, one at a border, the query's own), so that a lost or foreign row shows at full size."""
    from blok_b200 import lib
    if core == "mma":
        monkeypatch.setenv("BLOK_MLA_ATTEND_IMPL", "mma")
    rng = np.random.default_rng(H + rank)
    n, page = 1000, 64
    pos = [0, 1, 62, 63, 64, 65, 127, 128, 129, 500, 640, 998, 999]
    rows = rng.normal(size=(n, rank + rot)).astype(np.float32) * 0.3
    q = rng.normal(size=(len(pos), H, rank + rot)).astype(np.float32) * 0.3
    for i, p in enumerate(pos):
        star = [p, 0, p // 2, max(0, p - 64), min(p, 63)][i % 5]
        q[i] += rows[star] * 4
    tq = torch.from_numpy(q).to(cuda).to(dtype)
    tr = torch.from_numpy(rows).to(cuda).to(dtype)
    pool, table = paged(tr, page, 3, cuda)
    slot = torch.full((len(pos),), 2, dtype=torch.int32, device=cuda)
    got = f64(lib.latent_attend(tq, pool, table, slot, torch.tensor(pos, dtype=torch.int32, device=cuda), rank, 0.5, n))
    want = attend_plain(f64(tq), f64(tr), rank, 0.5, pos)
    bar = 1e-5 if dtype == torch.float32 else 5e-3  # bf16: the output's own rounding
    for i, p in enumerate(pos):
        assert np.max(np.abs(got[i] - want[i])) < bar * np.abs(want[i]).max(), p


@pytest.mark.parametrize("H,dim,rot,dv", [(1, 32, 32, 16), (3, 64, 32, 64), (2, 64, 64, 128), (2, 128, 64, 112), (2, 192, 64, 256),
                                             (2, 128, 64, 128), (3, 64, 64, 64), (1, 192, 64, 128)])
@pytest.mark.parametrize("T,n", [(33, 33), (200, 200), (64, 321), (129, 128 + 129), (40, 1000)])
def test_latent_prompt(cuda, H, dim, rot, dv, T, n):
    from blok_b200 import lib
    rng = np.random.default_rng(H + dim + T)
    q = rng.normal(size=(T, H, dim + rot)).astype(np.float32) * 0.3
    kv = rng.normal(size=(n, H * (dim + dv))).astype(np.float32)
    kr = rng.normal(size=(n, rot)).astype(np.float32)
    for i in range(0, T, 3):  # one key stands out: the query's own, the first, one in the middle, one at a tile's edge
        p = n - T + i
        star = [p, 0, p // 2, p // 64 * 64, max(0, p // 64 * 64 - 1)][(i // 3) % 5]
        q[i, :, dim:] += kr[star] * 2.5
    q, kv, kr = (plain.bf16_round(a) for a in (q, kv, kr))
    got = f64(lib.latent_prompt(bf16(q, cuda), bf16(kv, cuda), bf16(kr, cuda), dim, dv, 0.4)).reshape(T, H, dv)
    k = np.concatenate([kv[:, :H * dim].reshape(n, H, dim), np.repeat(kr[:, None], H, axis=1)], axis=2).astype(np.float64)
    v = kv[:, H * dim:].reshape(n, H, dv).astype(np.float64)
    s = np.einsum("ihd,jhd->hij", q.astype(np.float64), k) * 0.4
    s = np.where(np.arange(n)[None, None] <= (n - T + np.arange(T))[None, :, None], s, -np.inf)
    w = np.exp(s - s.max(axis=-1, keepdims=True))
    want = np.einsum("hij,jhd->ihd", w / w.sum(axis=-1, keepdims=True), v)
    err = np.abs(got - want).max(axis=(1, 2)) / np.abs(want).max()
    assert err.max() < 5e-3, (int(err.argmax()), err.max())


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
    """Every layer run's residual and every logit of a prompt, then the same tokens in portions and one by one."""
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
        assert_rows(run[i], layers[i], dtype, "after layer run %d" % i)
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
def test_prompts_longer_than_a_chunk_and_long_decoding(cuda, folder, dtype):
    from blok_b200 import lib
    d, cfg, tensors = folder("mixed")
    tok = tokens_of(cfg, 420, 6)
    model = lib.Model.open(d, dtype=dtype, max_ctx=420, prefill_chunk=96)
    got = np.concatenate([model.extend(0, tok[:230], range(230)), feed(model, 0, tok[230:], [1])])
    assert_rows(got, plain.forward(cfg, tensors, tok), dtype)
    model.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_key_decides(cuda, tmp_path, dtype):
    """One far token answers the last query (sharp queries): exchanging it must move the last logits as the plain evaluation
    says, from a prompt and from decoding alike."""
    from blok_b200 import lib

    def sharpen(cfg, t):
        t["l0.mix.uq"] = plain.bf16_round(t["l0.mix.uq"] * 4)
    cfg, tensors = cases.write(str(tmp_path), "latent", seed=8, edit=sharpen)
    T = 210
    tok = np.random.default_rng(11).integers(0, cfg["vocab"], T)
    base, most = plain.forward(cfg, tensors, tok)[-1], (0.0, None, None)
    for far in range(60):
        other = tok.copy()
        other[far] = (tok[far] + 1) % cfg["vocab"]
        moved = plain.forward(cfg, tensors, other)[-1] - base
        if moved.std() > most[0]:
            most = (moved.std(), other, moved)
    assert most[0] > 0.3 * base.std(), "a far token matters"
    model = lib.Model.open(str(tmp_path), dtype=dtype, max_batch=3, max_ctx=256, kv_page_rows=32)
    for sizes in ([T], [T - 1, 1], [64, 1]):
        got = []
        for x in (tok, most[1]):
            got.append(feed(model, 1, x.tolist(), sizes)[-1])
            model.release_slot(1)
        bar = TIGHT if dtype == "float32" else 0.2
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
            nxt = model.step_slots(slots, torch.tensor(ids, dtype=torch.int32, device=cuda))
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


def test_generation_through_the_scheduler(cuda, folder, tmp_path):
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
    for edit, message in ((lambda c, t: t.pop("l1.mix.dkv.norm"), "missing tensor l1.mix.dkv.norm"),
                          (lambda c, t: t.__setitem__("head", t["head"][:-1]), "tensor head has another type, shape or size"),
                          (lambda c, t: t.__setitem__("l0.mlp.table", t["l0.mlp.table"] + 5), "l0.mlp.table names expert")):
        cases.write(str(tmp_path), "mixed", edit=edit)
        with pytest.raises(lib.BlokError, match=message):
            lib.Model.open(str(tmp_path))
