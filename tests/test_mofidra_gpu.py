"""The Mofidra design in the engine against tests/plain_mofidra.py (float64, whole sequences, one
function per mechanism, no cache).  Every test makes its own small model (tests/mofidra_util.py).

Covered: differential attention and each feed-forward alone; whole prompts against token-by-token
stepping; portions of changing size down to two tokens; batches of unequal requests against each
alone; pages and slots given back and used again; keys far back, at page borders and among the first
tokens with one score made to stand out in either map; long portions beside single tokens; long
decoding; other sizes, also counts of one and sizes that are equal; the single kernels (attention in
all its launch shapes, preparation of heads in two parts, router, ungated experts, products with an
activation, a norm behind two sublayers) against the plain functions; greedy generation through the
engine's entry point, the command line and the trace runner.
"""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import mofidra_util as U
import plain_mofidra as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
F64 = torch.float64
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _setup(tmp_path, cfg, seed, **kw):
    W = U.make_weights(cfg, seed, **kw)
    return W, U.write_model(str(tmp_path / f"m{seed}"), cfg, W)


# ----------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
def test_each_mechanism_alone(tmp_path, dtype):
    cases = [(None, {}), ("dense", {}), ("moe", {}),
             (None, dict(heads=4, kv=4, dim=32, vdim=32, diff=0.8, rot=None)),
             (None, dict(heads=5, kv=1, dim=10, vdim=14, diff=0.05, rot=(4, 30.0), scale=0.7)),
             ("moe", dict(heads=3, kv=3, dim=64, vdim=128, experts=9, top=3, shared=None)),
             ("moe", dict(heads=2, kv=1, dim=16, vdim=200, experts=4, top=1, shared=5)),
             ("dense", dict(heads=1, kv=1, dim=128, vdim=16, emb=7.0, rot=(128, 77.0), loop=(0, 1, 3)))]
    for n, (mlp, kw) in enumerate(cases):
        cfg = U.single(mlp, **kw)
        W, path = _setup(tmp_path, cfg, 100 + n)
        toks = U.tokens_for(cfg, 77, n)
        want = U.plain_logits(cfg, W, toks)
        r = U.make_runner(path, dtype, pages=8)
        whole = U.run_cuts(r, "w", toks, [77])
        assert U.close(whole, want, dtype), (mlp, kw, U.rel_err(whole, want))
        stepped = U.run_cuts(r, "s", toks, [1] * 77)             # the same slot and pages once more
        assert U.close(stepped, want, dtype), (mlp, kw, "token by token", U.rel_err(stepped, want))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix_a", "mix_b", "mix_c"])
def test_portions_of_any_size(tmp_path, dtype, name, n=150):
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 7)
    toks = U.tokens_for(cfg, n, 3)
    want = U.plain_logits(cfg, W, toks)
    r = U.make_runner(path, dtype, pages=12)
    ragged, pattern = [], [2, 15, 1, 16, 17, 31, 2, 2, 33, 5]
    while sum(ragged) < n:
        ragged.append(min(pattern[len(ragged) % len(pattern)], n - sum(ragged)))
    for cuts in ([n], [n - 40] + [1] * 40, ragged, [16] * (n // 16) + [n % 16], [2] * (n // 2), [3] * (n // 3), [130, 2, 18]):
        cuts = [c for c in cuts if c]
        got = U.run_cuts(r, "p", toks, cuts)
        assert U.close(got, want, dtype), (cuts[:6], U.rel_err(got, want))
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_portions_beside_single_tokens(tmp_path, dtype, name="mix_b"):
    """Portions of 140 to 300 tokens in one step with another request's single token, the single token
    before the portion and after it, against the plain model of each request alone."""
    from llm_singularity_b200.engine.batch import StepEntry
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 13)
    x, y = U.tokens_for(cfg, 450, 6), U.tokens_for(cfg, 170, 7)
    want_x, want_y = U.plain_logits(cfg, W, x), U.plain_logits(cfg, W, y)
    r = U.make_runner(path, dtype, pages=48)
    assert r.open("x") and r.open("y")
    every = lambda n: list(range(n))
    a = r.step([StepEntry("y", y[:139], every(139))]).float().cpu()
    b = r.step([StepEntry("y", y[139:140], [0]), StepEntry("x", x[:300], every(300))]).float().cpu()
    c = r.step([StepEntry("x", x[300:440], every(140)), StepEntry("y", y[140:141], [0])]).float().cpu()
    d = r.step([StepEntry("y", y[141:], every(29)), StepEntry("x", x[440:], every(10))]).float().cpu()
    r.close("x"); r.close("y")
    r.check_kernels()
    got_x = torch.cat([b[1:], c[:140], d[29:]])
    got_y = torch.cat([a, b[:1], c[140:], d[:29]])
    assert U.close(got_x, want_x, dtype), U.rel_err(got_x, want_x)
    assert U.close(got_y, want_y, dtype), U.rel_err(got_y, want_y)
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix_a", "mix_b", "mix_c"])
def test_mixed_batches_with_slots_and_pages_used_again(tmp_path, dtype, name):
    """Four requests of unequal length stepped together (portions beside single tokens, a request
    left out of some steps, ends at different times, a fifth request taking over a freed slot and
    freed pages) against the plain model of each alone."""
    from llm_singularity_b200.engine.batch import StepEntry
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 9)
    lens = {"a": 70, "b": 23, "c": 41, "d": 1, "e": 37}
    toks = {k: U.tokens_for(cfg, n, 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: U.plain_logits(cfg, W, t) for k, t in toks.items()}
    r = U.make_runner(path, dtype, pages=10, slots=4)      # 160 token places for 172 tokens
    plan = [[("a", 33), ("b", 2)], [("a", 1), ("b", 17), ("c", 5)], [("d", 1), ("c", 1), ("a", 1)],
            [("b", 1), ("c", 30), ("a", 20)], [("b", 1), ("a", 1), ("c", 1)], [("b", 1), ("c", 2)],
            [("b", 1), ("a", 14), ("c", 2)], [("e", 36)], [("e", 1)]]
    at = {k: 0 for k in lens}
    got = {k: [] for k in lens}
    for step in plan:
        entries, who = [], []
        for k, n in step:
            n = min(n, lens[k] - at[k])
            if n <= 0:
                continue
            if not r.cache.has(k):
                assert r.open(k), f"no slot for {k}"
            entries.append(StepEntry(k, toks[k][at[k]:at[k] + n], list(range(n))))
            who.append((k, n))
        logits = r.step(entries).float().cpu()
        row = 0
        for k, n in who:
            got[k].append(logits[row:row + n].clone())
            row += n
            at[k] += n
            if at[k] == lens[k]:
                r.close(k)
    r.check_kernels()
    assert at == lens
    for k in lens:
        assert U.close(torch.cat(got[k]), want[k], dtype), (k, U.rel_err(torch.cat(got[k]), want[k]))
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_page_borders_and_first_tokens(tmp_path, dtype):
    """A strongly peaked softmax in both maps against pages of 16: a key that is lost, one page or one
    place off, or a first token left out changes the logits by far more than the tolerance."""
    for kw, seed in ((dict(), 31), (dict(heads=4, kv=4, dim=64, vdim=64, rot=(64, 1e4), diff=0.7), 32),
                     (dict(heads=8, kv=2, dim=16, vdim=96, rot=None), 33)):
        cfg = U.single(mlp=None, **kw)
        W, path = _setup(tmp_path, cfg, seed, sharpen=3.0)
        n = 300
        toks = U.tokens_for(cfg, n, 5)
        want = U.plain_logits(cfg, W, toks)
        r = U.make_runner(path, dtype, pages=20)
        for cuts in ([n], [255, 1, 1, 15, 17, 11], [n - 64] + [1] * 64, [49, 2, 48, 1, 1, 49, 50, 100], [129, 2, 130, 39]):
            got = U.run_cuts(r, "f", toks, cuts)
            assert U.close(got, want, dtype), (kw, cuts[:4], U.rel_err(got, want))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path, dtype, name="mix_b"):
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 13)
    n = 200
    toks = U.tokens_for(cfg, n, 8)
    want = U.plain_logits(cfg, W, toks)
    r = U.make_runner(path, dtype, pages=14)
    got = U.run_cuts(r, "l", toks, [3] + [1] * (n - 3))
    assert U.close(got, want, dtype), U.rel_err(got, want)
    assert r.graph_replays > 150                              # single tokens replay a captured step


@pytest.mark.parametrize("dtype", DTYPES)
def test_sublayers_on_two_streams_give_the_same_bits(tmp_path, dtype, monkeypatch, name="mix_b"):
    """A step of few rows runs mixer and feed-forward on two streams (captured in a graph and not): the same
    bits as one after the other, over many steps whose buffers are reused."""
    from llm_singularity_b200 import kernels as K
    from llm_singularity_b200.engine.batch import StepEntry
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 41)
    toks = {k: U.tokens_for(cfg, 90, 50 + i) for i, k in enumerate("abc")}
    got = []
    for limit in (0, 64):
        monkeypatch.setattr(K, "OVERLAP_SUBLAYERS", limit)
        r = U.make_runner(path, dtype, pages=24)
        assert all(r.open(k) for k in toks)
        rows = [r.step([StepEntry(k, t[:20], [19]) for k, t in toks.items()]).float().cpu()]
        rows += [r.step([StepEntry(k, t[i:i + 1], [0]) for k, t in toks.items()]).float().cpu() for i in range(20, 80)]
        rows.append(r.step([StepEntry("b", toks["b"][80:], [9]), StepEntry("a", toks["a"][80:81], [0])]).float().cpu())
        r.check_kernels()
        assert r.graph_replays > 40
        got.append(torch.cat(rows))
    assert torch.equal(got[0], got[1])


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(tmp_path, dtype, name="mix_a"):
    """Greedy generation through Engine (scheduler, portions of 16, three requests at once) gives
    the tokens the plain model picks, wherever its choice is not a near tie."""
    from llm_singularity_b200 import Engine
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 17)
    eng = Engine(path, dtype=dtype, kv_block_size=16, num_kv_blocks=24, max_batch_size=3,
                 max_tokens_per_batch=48, prefill_chunk=16)
    prompts = [U.tokens_for(cfg, n, 40 + n) for n in (5, 37, 18)]
    new = 12
    ids = [eng.add_request(p, max_new_tokens=new) for p in prompts]
    out = {i: [] for i in ids}
    while eng.has_work():
        for rid, tok, _ in eng.step():
            assert tok >= 0
            out[rid].append(tok)
    clear = 0
    for rid, p in zip(ids, prompts):
        seq = list(p)
        for tok in out[rid]:
            logits = U.plain_logits(cfg, W, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if (top2[0] - top2[1]) > (0.05 if dtype == "float32" else 0.4):
                assert tok == int(logits.argmax()), (rid, len(seq))
                clear += 1
            seq.append(tok)
        assert len(out[rid]) == new
    assert clear > new


def test_requests_share_the_pages_of_a_common_prefix(tmp_path, name="mix_b"):
    """Every cache of the design is full pages, a looped layer's passes included, so a second request with the
    same first tokens takes them from the prefix tree and generates what the plain model picks."""
    from llm_singularity_b200 import Engine
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 37)
    eng = Engine(path, dtype="float32", kv_block_size=16, num_kv_blocks=32, max_batch_size=2, max_tokens_per_batch=64)
    assert eng.prefix is not None
    common = U.tokens_for(cfg, 40, 3)
    for k, tail in enumerate(([5, 9, 2], [7, 1])):
        rid = eng.add_request(common + tail, max_new_tokens=5)
        seq = common + tail
        while eng.has_work():
            for r, tok, _ in eng.step():
                assert r == rid
                top2 = torch.topk(U.plain_logits(cfg, W, seq)[-1], 2)
                if top2.values[0] - top2.values[1] > 0.05:
                    assert tok == int(top2.indices[0]), (k, len(seq))
                seq.append(tok)
        assert eng.prefix.hits == 2 * k


# ----------------------------------------------------------------- kernels against plain functions
def _ctx(q_lens, kv_lens, rows=None):
    from llm_singularity_b200.engine.batch import ContextBuilder
    b = ContextBuilder("cuda", 4096, 64)
    ctx, _ = b.build([[0] * n for n in q_lens], [kv - q for kv, q in zip(kv_lens, q_lens)],
                     rows or list(range(len(q_lens))), [[] for _ in q_lens])
    ctx._keep = b
    return ctx


def _pages(slots, max_kv, nkv, dk, dv, page, dtype, seed=0):
    from llm_singularity_b200.parts import KVCacheView
    per = -(-max_kv // page)
    n = slots * per + 3
    perm = torch.randperm(n, generator=torch.Generator().manual_seed(seed))[:slots * per].view(slots, per)
    return KVCacheView(torch.zeros(n, nkv, page, dk, dtype=dtype, device="cuda"),
                       torch.zeros(n, nkv, page, dv, dtype=dtype, device="cuda"),
                       perm.to(torch.int32).cuda(), page, None, 0)


def _fill(cache, row, K, V):
    pos = torch.arange(K.shape[0])
    pages = cache.block_table[row].cpu()[pos // cache.page_size].long()
    cache.k_pages[pages, :, pos % cache.page_size, :] = K.to(cache.k_pages.dtype).cuda()
    cache.v_pages[pages, :, pos % cache.page_size, :] = V.to(cache.v_pages.dtype).cuda()


def _difference(q, Kd, Vd, pos_q, scale, lam, eps, post, window=0, chunk=0):
    """q [n, heads, 2, dk], Kd [kv, nkv, 2, dk], Vd [kv, nkv, dv] in float64 -> [n, heads, dv]."""
    n, nh = q.shape[:2]
    kv, nkv = Kd.shape[:2]
    pos_k = torch.arange(kv)
    seen = pos_k[None, :] <= pos_q[:, None]
    if window:
        seen &= pos_k[None, :] > pos_q[:, None] - window
    if chunk:
        seen &= pos_k[None, :] >= (pos_q[:, None] // chunk) * chunk
    out = torch.zeros(n, nh, Vd.shape[-1], dtype=F64)
    for h in range(nh):
        g = h // (nh // nkv)
        a = [torch.softmax((q[:, h, m] @ Kd[:, g, m].T * scale).masked_fill(~seen, float("-inf")), -1) @ Vd[:, g] for m in (0, 1)]
        out[:, h] = P.unit_rms(a[0] - lam * a[1], eps) * post
    return out


@pytest.mark.parametrize("dtype, shape", [(torch.float32, 0)] + [(torch.bfloat16, s) for s in (0, 1, 2, 3, 4, 5, 7, 12)])    # (32-bit has one shape)
@pytest.mark.parametrize("nh, nkv, dk, dv, window, chunk, page", [
    (4, 2, 32, 16, 0, 0, 16), (6, 2, 96, 56, 0, 0, 16), (3, 3, 10, 14, 0, 0, 8), (4, 1, 64, 128, 0, 0, 16), (2, 2, 128, 256, 0, 0, 32),
    (8, 2, 64, 64, 40, 0, 16), (8, 8, 40, 72, 0, 48, 16), (2, 1, 24, 200, 33, 64, 16), (4, 4, 64, 128, 70, 0, 16)])
def test_differential_attention_kernel_one_score_standing_out(dtype, nh, nkv, dk, dv, window, chunk, page, shape, monkeypatch):
    """Three requests in one launch (a single token, a prompt portion, a whole prompt).  All keys are alike
    but one per map and request, which every query of that map scores high: far back, on a page border,
    first in the sequence, last, and around the window's and the chunk's edge.  Every launch shape."""
    from llm_singularity_b200 import kernels as K
    monkeypatch.setattr(K, "DV_BLOCK_SHAPE", shape)
    g = torch.Generator().manual_seed(dk + dv)
    q_lens, kv_lens = ([1, 37, 170], [131, 90, 170]) if shape != 3 else ([37, 1, 170], [90, 131, 170])
    slot_rows = [0, 2, 1]
    ctx = _ctx(q_lens, kv_lens, rows=slot_rows)
    scale, lam, eps, post = 1.0 / math.sqrt(dk), 0.6, 1e-5, 0.7
    mixing = torch.tensor([lam], device="cuda")
    edge = [max(kv - 1 - (window or 40) + d, 0) for kv in kv_lens for d in (0, 1)]
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    for t0, t1 in (([3, 0, 15], [16, 64, 48]), ([0, 79, 0], [89, 89, 169]), (edge[0::2], edge[1::2]), (edge[1::2], edge[0::2]),
                   ([48, 47, 96], [47, 48, 95])):
        cache = _pages(3, 176, nkv, 2 * dk, dv, page, dtype, seed=1)
        qs, want = [], []
        for r, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
            Kd = 0.1 * torch.randn(kv, nkv, 2, dk, generator=g)
            Kd[min(t0[r], kv - 1), :, 0, 0] = 6.0
            Kd[min(t1[r], kv - 1), :, 1, 0] = 6.0
            Vd = torch.randn(kv, nkv, dv, generator=g)
            q = 0.1 * torch.randn(ql, nh, 2, dk, generator=g)
            q[..., 0] = 1.5 / scale
            Kd, Vd, q = (t.to(dtype).double() for t in (Kd, Vd, q))
            _fill(cache, slot_rows[r], Kd.reshape(kv, nkv, 2 * dk), Vd)
            want.append(_difference(q, Kd, Vd, torch.arange(kv - ql, kv), scale, lam, eps, post, window, chunk))
            qs.append(q)
        T = sum(q_lens)
        q = torch.cat(qs).reshape(T, nh * 2 * dk).to(dtype).cuda()
        out = torch.zeros(T, nh * dv, dtype=dtype, device="cuda")
        K.attention_diff(q, nh, nkv, dk, dv, ctx, cache, scale, window, chunk, mixing, eps, post, out)
        err = (out.double().cpu() - torch.cat(want).reshape(T, nh * dv)).abs().max()
        assert err <= tol, (t0, t1, err)
    K.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, dk, dv", [(4, 2, 64, 128), (2, 1, 64, 64), (3, 3, 128, 128), (2, 2, 48, 80)])
@pytest.mark.parametrize("window", [0, 150])
def test_differential_attention_of_long_portions(dtype, nh, nkv, dk, dv, window):
    """Portions of 128 tokens and more (a kernel of their own where sizes allow) behind cached tokens, of
    unequal length, after single tokens: random values and a key per map that stands out."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(dk * dv)
    q_lens, kv_lens = [1, 1, 200, 131], [300, 17, 333, 131]
    ctx = _ctx(q_lens, kv_lens, rows=[3, 0, 2, 1])
    scale, lam, eps, post = 1.0 / math.sqrt(dk), 0.8, 1e-6, 0.4
    mixing = torch.tensor([lam], device="cuda")
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    for t0, t1 in (([0, 0, 0, 0], [299, 16, 132, 64]), ([150, 16, 190, 63], [151, 3, 131, 128]), ([149, 1, 183, 0], [150, 2, 182, 1])):
        cache = _pages(4, 336, nkv, 2 * dk, dv, 16, dtype, seed=4)
        qs, want = [], []
        for r, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
            Kd, Vd = 0.5 * torch.randn(kv, nkv, 2, dk, generator=g), torch.randn(kv, nkv, dv, generator=g)
            q = 0.5 * torch.randn(ql, nh, 2, dk, generator=g)
            Kd[t0[r], :, 0, 0] = 4.0
            Kd[t1[r], :, 1, 0] = 4.0
            q[..., 0] = 1.5 / scale
            Kd, Vd, q = (t.to(dtype).double() for t in (Kd, Vd, q))
            _fill(cache, [3, 0, 2, 1][r], Kd.reshape(kv, nkv, 2 * dk), Vd)
            want.append(_difference(q, Kd, Vd, torch.arange(kv - ql, kv), scale, lam, eps, post, window))
            qs.append(q)
        T = sum(q_lens)
        q = torch.cat(qs).reshape(T, nh * 2 * dk).to(dtype).cuda()
        out = torch.zeros(T, nh * dv, dtype=dtype, device="cuda")
        K.attention_diff(q, nh, nkv, dk, dv, ctx, cache, scale, window, 0, mixing, eps, post, out)
        err = (out.double().cpu() - torch.cat(want).reshape(T, nh * dv)).abs().max()
        assert err <= tol, (t0, t1, err)
    K.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh, nkv, dk, dv, rot", [(4, 2, 24, 40, 16), (3, 1, 10, 14, 10), (2, 2, 64, 128, 0)])
def test_preparation_of_heads_in_two_parts(dtype, nh, nkv, dk, dv, rot):
    """Both parts of every query and key head are rotated as heads of their own, at far positions too, and
    a key's parts lie side by side in its cache row."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(dk)
    q_lens, kv_lens = [3, 1, 20], [40, 130, 20]
    ctx = _ctx(q_lens, kv_lens)
    cache = _pages(3, 144, nkv, 2 * dk, dv, 16, dtype)
    T, cols = sum(q_lens), 2 * nh * dk + 2 * nkv * dk + nkv * dv
    proj = torch.randn(T, cols, generator=g).to(dtype)
    pos = torch.cat([torch.arange(kv - ql, kv) for ql, kv in zip(q_lens, kv_lens)])
    d = proj.double()
    q, k, v = d[:, :2 * nh * dk].view(T, nh, 2, dk), d[:, 2 * nh * dk:2 * (nh + nkv) * dk].view(T, nkv, 2, dk), d[:, 2 * (nh + nkv) * dk:]
    kw = {}
    if rot:
        q, k = P.turn_halves(q, pos, rot, 500.0), P.turn_halves(k, pos, rot, 500.0)
        inv = torch.tensor([500.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32, device="cuda")
        kw = dict(inv_freq=inv, rotary_dim=rot)
    out = torch.empty(T, 2 * nh * dk, dtype=dtype, device="cuda")
    K.attention_prep(proj.cuda(), 0, 2 * nh * dk, 2 * (nh + nkv) * dk, nh, nkv, dk, dv, ctx, cache, out, maps=2, **kw)
    tol = 5e-5 if dtype == torch.float32 else 2e-2
    assert (out.double().cpu() - q.reshape(T, -1)).abs().max() < tol
    at = 0
    for r, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
        p = torch.arange(kv - ql, kv)
        page = cache.block_table[r].cpu()[p // 16].long()
        kc, vc = cache.k_pages.cpu()[page, :, p % 16].double(), cache.v_pages.cpu()[page, :, p % 16].double()
        assert (kc - k[at:at + ql].reshape(ql, nkv, 2 * dk)).abs().max() < tol
        assert (vc - v[at:at + ql].reshape(ql, nkv, dv)).abs().max() == 0
        at += ql
    K.check_status()


@pytest.mark.parametrize("E, top", [(5, 2), (12, 3), (3, 1), (40, 4), (2, 2)])
def test_router_with_bias_in_the_logits(E, top):
    """The bias changes choices and weights; the weights are the softmax over the chosen logits alone.  Large
    logits do not overflow."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(E)
    T = 64
    z, b = 2.0 * torch.randn(T, E, generator=g), 2.0 * torch.randn(E, generator=g)
    z[5] += 300.0
    ids, wts = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, dtype=torch.float32, device="cuda")
    K.moe_route(z.cuda(), top, "softmax_chosen", False, ids, wts, choice_bias=b.cuda(), bias_in_logits=True)
    want_ids, want = P.choose(z.double() + b.double(), top)
    assert torch.equal(ids.cpu().long(), want_ids)
    if top < E:
        assert not torch.equal(want_ids, P.choose(z.double(), top)[0])
    tol = torch.where(torch.arange(T) == 5, 1e-4, 2e-6)[:, None]                # (300 + x keeps fewer digits of x)
    assert ((wts.double().cpu() - want).abs() < tol).all()
    K.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W, F, E, top, S", [(5, 64, 48, 6, 2, 40), (300, 64, 48, 6, 2, 40), (33, 52, 18, 4, 3, 0), (1, 128, 64, 9, 1, 8),
                                                (700, 136, 264, 5, 2, 72)])
def test_ungated_experts_beside_a_shared_one(dtype, T, W, F, E, top, S):
    """The routed feed-forward as a part against the plain one: few tokens (choosing inside the sorting
    kernel) and many, sizes for the tensor-core products and others."""
    from llm_singularity_b200.config.specs import DenseMLPSpec, MoESpec
    from llm_singularity_b200.parts import FEED_FORWARDS, Runtime
    g = torch.Generator().manual_seed(T + W)
    Wt = {"router": 3.0 * torch.randn(E, W, generator=g) / math.sqrt(W), "router.b": torch.randn(E, generator=g)}
    for e in range(E):
        Wt[f"e{e}.up"] = torch.randn(F, W, generator=g) / math.sqrt(W)
        Wt[f"e{e}.down"] = torch.randn(W, F, generator=g) / math.sqrt(F)
    mlp = {"kind": "moe", "router": {"experts": E, "top": top}}
    if S:
        Wt.update({"shared.up": torch.randn(S, W, generator=g) / math.sqrt(W), "shared.down": torch.randn(W, S, generator=g) / math.sqrt(S),
                   "shared.sg": 2.0 * torch.randn(1, W, generator=g) / math.sqrt(W)})
        mlp["shared"] = {"ff": S}
    Wt = {n: t.to(torch.bfloat16) for n, t in Wt.items()}
    h = torch.randn(T, W, generator=g).to(torch.bfloat16)
    want = P.routed(h.double(), {n: t.double() for n, t in Wt.items()}, "", mlp)
    rt = Runtime("cuda", dtype)
    shared = DenseMLPSpec(hidden_size=W, intermediate_size=S, activation="relu_squared") if S else None
    part = FEED_FORWARDS.build(MoESpec(hidden_size=W, expert_size=F, num_experts=E, top=top, activation="relu_squared",
                                       score="softmax_chosen", weight_on="output", gated=False, router_bias=True, shared=shared,
                                       shared_gate=bool(S)), rt)
    dev = lambda n, vec=False: Wt[n].to("cuda", torch.float32 if vec else dtype)
    own = {"router": dev("router"), "router_bias": dev("router.b", True)}
    own.update({f"e{e}.{w}": dev(f"e{e}.{w}") for e in range(E) for w in ("up", "down")})
    if S:
        own["shared_gate"] = dev("shared.sg")
        part.children()["shared"].load({"up_proj": dev("shared.up"), "down_proj": dev("shared.down")})
    part.load(own)
    got = part.forward(h.to("cuda", dtype), None).double().cpu()
    scale = want.pow(2).mean().sqrt()
    assert (got - want).abs().max() < (1e-5 if dtype == torch.float32 else 5e-2) * max(1.0, scale), (got - want).abs().max()


@pytest.mark.parametrize("tile", [16, 32, 64, 128])
@pytest.mark.parametrize("act", ["relu_squared", "silu", "capped_glu"])
@pytest.mark.parametrize("T, H, F, E, top", [(3, 64, 40, 4, 2), (150, 128, 136, 5, 3), (9, 72, 264, 9, 1)])
def test_grouped_products_over_row_tiles_of_any_height(tile, act, T, H, F, E, top, monkeypatch):
    """Experts gated and not, through both orientations of the grouped product; one expert gets more rows than a
    tile, another none."""
    from llm_singularity_b200 import kernels as K
    monkeypatch.setattr(K, "MOE_ROW_TILE", tile)
    g = torch.Generator().manual_seed(T + F)
    gated, limit = act != "relu_squared", 0.9
    bf = lambda *shape: (torch.randn(*shape, generator=g) / math.sqrt(shape[-1])).to(torch.bfloat16)
    up, gate, down = bf(E, F, H), bf(E, F, H), bf(E, H, F)
    x = torch.randn(T, H, generator=g).to(torch.bfloat16)
    ids = torch.stack([torch.randperm(E - 1, generator=g)[:top] for _ in range(T)])          # the last expert idles
    ids[:2 * T // 3, 0] = 1
    wts = torch.rand(T, top, generator=g) + 0.2
    want = torch.zeros(T, H, dtype=F64)
    for t in range(T):
        for k in range(top):
            e = int(ids[t, k])
            u, z = up[e].double() @ x[t].double(), gate[e].double() @ x[t].double()
            if act == "capped_glu":
                z = torch.clamp(z, max=limit)
                hid = z * torch.sigmoid(1.702 * z) * (torch.clamp(u, -limit, limit) + 1.0)
            else:
                hid = z * torch.sigmoid(z) * u if gated else P.relu_squared(u)
            want[t] += wts[t, k].double() * (down[e].double() @ hid)
    w = torch.stack([gate, up], dim=2).reshape(E, 2 * F, H).contiguous() if gated else up
    out = torch.empty(T, H, dtype=torch.bfloat16, device="cuda")
    K.moe_experts(x.cuda(), ids.to(torch.int32).cuda(), wts.cuda(), w.cuda(), down.cuda(), act, "output", out, gated=gated,
                  limit=limit if act == "capped_glu" else 0.0)
    assert (out.double().cpu() - want).abs().max() < 3e-2 * max(1.0, want.abs().max())
    K.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("act", ["gelu_tanh", "relu_squared", "silu"])
@pytest.mark.parametrize("M, K_, N", [(1, 64, 40), (9, 128, 300), (16, 192, 1000), (40, 128, 264), (100, 1024, 128), (300, 64, 520), (700, 72, 130),
                                      (257, 4096, 256), (20, 52, 33)])
def test_product_with_an_activation_on_every_element(dtype, act, M, K_, N):
    """Through every product kernel that knows ungated activations (a few rows, tiles in both orientations, K
    split over a cluster, persistent blocks) and through the activation kernel behind the others."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(M + N)
    x = torch.randn(M, K_, generator=g).to(dtype)
    w = (1.5 * torch.randn(N, K_, generator=g) / math.sqrt(K_)).to(dtype)
    z = x.double() @ w.double().T
    want = {"gelu_tanh": P.gelu_tanh, "relu_squared": P.relu_squared, "silu": lambda t: t * torch.sigmoid(t)}[act](z)
    got = K.linear(x.cuda(), w.cuda(), plain_act=act).double().cpu()
    tol = 3e-5 if dtype == torch.float32 else 1.5e-2
    assert ((got - want).abs() <= tol * (1.0 + want.abs())).all(), (got - want).abs().max()
    K.check_status()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [52, 128, 2050, 4096, 5000])
def test_norm_behind_two_sublayers(dtype, hidden):
    """Both outputs join the 32-bit stream in one pass; the gathered form leaves the stream alone."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(hidden)
    T, eps = 11, 1e-5
    x = torch.randn(T, hidden, generator=g).cuda()
    a, b = torch.randn(T, hidden, generator=g).to(dtype).cuda(), (5.0 * torch.randn(T, hidden, generator=g)).to(dtype).cuda()
    w = torch.randn(hidden, generator=g).cuda()
    xd = x.double().cpu()
    stream = xd + a.double().cpu() + b.double().cpu()
    want = P.unit_rms(stream, eps) * w.double().cpu()
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    rows = torch.tensor([4, 0, 10, 4], dtype=torch.int32).cuda()
    picked = torch.empty(4, hidden, dtype=dtype, device="cuda")
    K.gather_add_rmsnorm(x, a, rows, w, eps, picked, delta2=b)
    assert torch.equal(x.double().cpu(), xd)
    assert (picked.double().cpu() - want[rows.cpu().long()]).abs().max() < tol
    out = torch.empty(T, hidden, dtype=dtype, device="cuda")
    K.add_rmsnorm(x, a, w, eps, out, delta2=b)
    assert (x.double().cpu() - stream).abs().max() < 1e-5
    assert (out.double().cpu() - want).abs().max() < tol
    K.check_status()


# ------------------------------------------------------------------------ as a user runs it
@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_user_runs_it(tmp_path, dtype):
    """bin/trace_run as a process of its own, fed step by step: seven requests through four slots
    and a pool smaller than their sum (mixed portions and single tokens), then each request in
    portions of changing size; every position against the plain model."""
    import cuttings
    import numpy as np
    import replay_util
    cfg = U.CONFIGS["mix_a"]
    W, path = _setup(tmp_path, cfg, 23)
    seqs = {f"q{i}": U.tokens_for(cfg, n, 60 + i) for i, n in enumerate((5, 70, 33, 1, 100, 64, 21))}
    want = {rid: U.plain_logits(cfg, W, t) for rid, t in seqs.items()}
    for k, (steps, max_tokens) in enumerate((cuttings.mixed(seqs, seed=3), cuttings.portions(seqs))):
        out = str(tmp_path / f"out{k}")
        replay_util.replay_subprocess(path, dtype, steps, out, max_tokens)
        rows = replay_util.collect(steps, out, cfg["vocab"])
        assert len(rows) == sum(len(t) for t in seqs.values())
        for rid, t in seqs.items():
            got = torch.from_numpy(np.stack([rows[(rid, p)] for p in range(len(t))]))
            assert U.close(got, want[rid], dtype), (k, rid, U.rel_err(got, want[rid]))


def test_command_line_serves_the_design(tmp_path):
    """bin/llm-serve-llama picks the design by config.json and generates greedily what the plain
    model picks (where its choice is clear)."""
    cfg = U.CONFIGS["mix_b"]
    W, path = _setup(tmp_path, cfg, 29)
    prompts = [U.tokens_for(cfg, n, 70 + n) for n in (4, 19)]
    (tmp_path / "p.json").write_text(json.dumps(prompts))
    cmd = [sys.executable, os.path.join(ROOT, "bin", "llm-serve-llama"), "--model-dir", path, "--dtype", "fp32",
           "--prompt-ids", str(tmp_path / "p.json"), "--max-new-tokens", "6", "--ignore-eos",
           "--num-kv-blocks", "16", "--max-batch-size", "2"]
    res = subprocess.run(cmd, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr
    outs = [json.loads(line)["tokens"] for line in res.stdout.splitlines()]
    assert len(outs) == 2 and all(len(o) == 6 for o in outs)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o:
            logits = U.plain_logits(cfg, W, seq)[-1]
            top2 = torch.topk(logits, 2).values
            if top2[0] - top2[1] > 0.05:
                assert tok == int(logits.argmax())
            seq.append(tok)
