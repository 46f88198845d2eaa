"""The Lilupel design in the engine against tests/plain_lilupel.py (float64, whole sequences, one function
per mechanism, no cache).  Every test makes its own small model (tests/lilupel_util.py).

Covered: each mixer and the routed feed-forward alone; whole prompts against token-by-token stepping;
portions of changing size down to two tokens; batches of unequal requests against each alone; pages and
slots given back and used again; keys just inside and just outside the window, at page borders and among
the first tokens with one score made to stand out; memories across the borders of chunks and
segments; long portions beside single tokens; long decoding; other sizes, also counts of one and sizes
that are equal; the single kernels against the plain functions; greedy generation through the engine's
entry point, the command line and the trace runner.
"""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import lilupel_util as U
import plain_lilupel as P

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
TYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def _setup(tmp_path, cfg, seed):
    W = U.make_weights(cfg, seed)
    return W, U.write_model(str(tmp_path / f"m{seed}"), cfg, W)


# ----------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", DTYPES)
def test_each_mechanism_alone(tmp_path, dtype):
    cases = [("parallel", dict(mlp=False)), ("parallel", {}), ("mamba2", dict(mlp=False)), ("mamba2", {}),
             ("parallel", dict(heads=4, kv=4, dim=64, vdim=64, window=20, rot=(64, 1e4), rheads=2, rdim=64, rvdim=64, rrot=(32, 50.0))),
             ("parallel", dict(heads=5, kv=1, dim=10, vdim=14, window=1, rot=(2, 30.0), rheads=1, rdim=6, rvdim=130, rrot=(6, 9.0), decay=[0.0])),
             ("parallel", dict(heads=2, kv=2, dim=128, vdim=128, window=300, rot=(64, 1e6), rheads=4, rdim=128, rvdim=8, rrot=(128, 1e6),
                               decay=[1.0, 0.999, 0.5, 0.9], left_scale=-0.5, right_scale=0.25)),
             ("mamba2", dict(heads=8, vdim=64, state=64, groups=1, conv=2, norm_groups=8)),
             ("mamba2", dict(heads=3, vdim=7, state=130, groups=3, conv=6, norm_groups=7)),
             ("mamba2", dict(heads=4, vdim=128, state=16, groups=2, conv=1, norm_groups=1, experts=9, top=5))]
    for n, (kind, kw) in enumerate(cases):
        cfg = U.single(kind, **kw)
        W, path = _setup(tmp_path, cfg, 100 + n)
        toks = U.tokens_for(cfg, 77, n)
        want = U.plain_logits(cfg, W, toks)
        r = U.make_runner(path, dtype, pages=8)
        whole = U.run_cuts(r, "w", toks, [77])
        assert U.close(whole, want, dtype), (kind, kw, U.rel_err(whole, want))
        stepped = U.run_cuts(r, "s", toks, [1] * 77)             # the same slot and pages once more
        assert U.close(stepped, want, dtype), (kind, kw, "token by token", U.rel_err(stepped, want))


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
    for cuts in ([n], [n - 40] + [1] * 40, ragged, [16] * (n // 16) + [n % 16], [2] * (n // 2), [3] * (n // 3), [130, 2, 18], [49, 48, 53]):
        cuts = [c for c in cuts if c]
        got = U.run_cuts(r, "p", toks, cuts)
        assert U.close(got, want, dtype), (cuts[:6], U.rel_err(got, want))
    r.cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix_a", "mix_b"])
def test_long_portions_beside_single_tokens(tmp_path, dtype, name):
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
def test_windows_page_borders_and_first_tokens(tmp_path, dtype):
    """A strongly peaked softmax against pages of 16 and windows around page borders: a key that is lost, or
    seen one place too long, changes the logits by far more than the tolerance.  Memories that hardly fade
    keep the first tokens in every logit."""
    for window, kw, seed in ((50, {}, 31), (64, dict(heads=4, kv=4, dim=64, vdim=64, rot=(64, 1e4)), 32), (17, dict(heads=8, kv=2, dim=16, vdim=96), 33),
                             (1000, dict(heads=2, kv=1, dim=128, vdim=128, rot=(128, 1e4), rdim=64, rvdim=64, rrot=(64, 1e4)), 34)):
        cfg = U.single("parallel", mlp=False, window=window, scale=12.0 / kw.get("dim", 24), decay=[1.0, 0.9995, 0.98], **kw)
        W, path = _setup(tmp_path, cfg, seed)
        n = 300
        toks = U.tokens_for(cfg, n, 5)
        want = U.plain_logits(cfg, W, toks)
        r = U.make_runner(path, dtype, pages=20)
        for cuts in ([n], [255, 1, 1, 15, 17, 11], [n - 64] + [1] * 64, [49, 2, 48, 1, 1, 49, 50, 100], [129, 2, 130, 39]):
            got = U.run_cuts(r, "f", toks, cuts)
            assert U.close(got, want, dtype), (window, kw, cuts[:4], U.rel_err(got, want))
    off = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], left=dict(cfg["layers"][0]["mixer"]["left"],
                                                                                                       mask={"size": 120})))])
    assert U.rel_err(U.plain_logits(off, W, toks), want) > 0.1


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix_a", "mix_b"])
def test_long_decoding(tmp_path, dtype, name):
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
def test_branches_on_two_streams_give_the_same_bits(tmp_path, dtype, monkeypatch, name="mix_b"):
    """A step of few rows runs the two mixers of a pair on two streams (captured in a graph and not): the same
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


def test_repeated_prompts_replay_their_graph(tmp_path, name="mix_b"):
    """A prompt of one length that comes again is captured and replayed (experts' places and scratch of the
    chunked memories included): the logits of different prompts stay those of the plain model."""
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 43)
    r = U.make_runner(path, "bfloat16", pages=24)
    for i in range(5):
        toks = U.tokens_for(cfg, 140, 90 + i)
        got = U.run_cuts(r, "g", toks, [140])
        assert U.close(got, U.plain_logits(cfg, W, toks), "bfloat16"), i
    assert r.graph_replays >= 2


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(tmp_path, dtype, name="mix_a"):
    """Greedy generation through Engine (scheduler, portions of 16, three requests at once) gives
    the tokens the plain model picks, wherever its choice is not a near tie."""
    from llm_singularity_b200 import Engine
    cfg = U.CONFIGS[name]
    W, path = _setup(tmp_path, cfg, 17)
    eng = Engine(path, dtype=dtype, kv_block_size=16, num_kv_blocks=24, max_batch_size=3,
                 max_tokens_per_batch=48, prefill_chunk=16)
    assert eng.prefix is None or not eng.prefix.hits               # states are not shared through a prefix tree
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
            if (top2[0] - top2[1]) > (0.01 if dtype == "float32" else 0.2) * float(logits.std()):
                assert tok == int(logits.argmax()), (rid, len(seq))
                clear += 1
            seq.append(tok)
        assert len(out[rid]) == new
    assert clear > new


# ----------------------------------------------------------------- kernels against plain functions
def _ctx(q_lens, kv_lens, rows=None, tokens=None):
    from llm_singularity_b200.engine.batch import ContextBuilder
    b = ContextBuilder("cuda", 4096, 64)
    ctx, _ = b.build(tokens or [[0] * n for n in q_lens], [kv - q for kv, q in zip(kv_lens, q_lens)],
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


@pytest.mark.parametrize("dtype, shape", [(torch.float32, 0)] + [(torch.bfloat16, s) for s in (0, 1, 2, 3, 4)])
@pytest.mark.parametrize("nh, nkv, dk, dv, window, page", [(4, 2, 32, 16, 33, 16), (6, 2, 96, 48, 64, 16), (3, 3, 10, 14, 21, 8),
                                                         (4, 1, 64, 64, 100, 16), (2, 2, 128, 128, 64, 32), (5, 5, 64, 128, 0, 16)])
def test_attention_with_a_learnt_sink_one_score_standing_out(dtype, nh, nkv, dk, dv, window, page, shape, monkeypatch):
    """Single tokens, a portion and a whole prompt in one launch.  All keys are alike but one, just inside the
    last row's window, just outside, far back, at a page border or first; sinks from negligible to above
    every score (those rows' weights all but vanish)."""
    from llm_singularity_b200 import kernels as K
    monkeypatch.setattr(K, "DV_BLOCK_SHAPE", shape)
    g = torch.Generator().manual_seed(dk + dv)
    q_lens, kv_lens, slots = [1, 1, 37, 170], [131, 9, 90, 170], [3, 0, 2, 1]
    ctx = _ctx(q_lens, kv_lens, rows=slots)
    scale = 1.0 / math.sqrt(dk)
    sink = torch.linspace(-4.0, 9.0, nh) if nh > 1 else torch.tensor([2.0])
    tol = 3e-5 if dtype == torch.float32 else 4e-2
    w = window or 1000
    for pick in (lambda kv: kv - w, lambda kv: kv - w - 1, lambda kv: 0, lambda kv: page - 1, lambda kv: page, lambda kv: kv - 1):
        cache = _pages(4, 176, nkv, dk, dv, page, dtype, seed=1)
        qs, want = [], []
        for r, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
            Kd = 0.1 * torch.randn(kv, nkv, dk, generator=g)
            Kd[min(max(pick(kv), 0), kv - 1), :, 0] = 5.0
            Vd = torch.randn(kv, nkv, dv, generator=g)
            q = 0.1 * torch.randn(ql, nh, dk, generator=g)
            q[..., 0] = 1.4 / scale
            Kd, Vd, q = (t.to(dtype).double() for t in (Kd, Vd, q))
            _fill(cache, slots[r], Kd, Vd)
            pos = torch.arange(kv)
            ok = P.in_window(pos, w)[kv - ql:]
            want.append(torch.stack([P.softmax_beside_sink(q[:, h] @ Kd[:, h // (nh // nkv)].T * scale, sink[h].double(), ok) @ Vd[:, h // (nh // nkv)]
                                     for h in range(nh)], dim=1))
            qs.append(q)
        T = sum(q_lens)
        q = torch.cat(qs).reshape(T, nh * dk).to(dtype).cuda()
        out = torch.zeros(T, nh * dv, dtype=dtype, device="cuda")
        K.attention_dv(q, nh, nkv, dk, dv, ctx, cache, scale, window, 0, None, out, sink=True, sink_logit=sink.cuda())
        err = (out.double().cpu() - torch.cat(want).reshape(T, nh * dv)).abs().max()
        assert err <= tol, err
    K.check_status()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("nh, nkv, dk, dv, rot", [(4, 2, 24, 40, 16), (3, 1, 10, 14, 10), (2, 2, 64, 128, 2)])
def test_preparation_with_heads_of_unit_rms(dtype, nh, nkv, dk, dv, rot):
    """Biases, heads of q and k of unit rms and turned (one head near zero: eps shows), at far positions too."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(dk)
    q_lens, kv_lens = [3, 1, 20], [40, 130, 20]
    ctx = _ctx(q_lens, kv_lens)
    cache = _pages(3, 144, nkv, dk, dv, 16, dtype)
    T, eps = sum(q_lens), 1e-3
    nq, nk, nv = nh * dk, nkv * dk, nkv * dv
    proj = torch.randn(T, nq + nk + nv, generator=g)
    bias = [torch.randn(n, generator=g) for n in (nq, nk, nv)]
    proj[:, :dk] = 0.01 * proj[:, :dk]
    bias[0][:dk] = 0.02
    proj = proj.to(dtype)
    d = proj.double()
    pos = torch.cat([torch.arange(kv - ql, kv) for ql, kv in zip(q_lens, kv_lens)])
    q, k = (d[:, :nq] + bias[0]).view(T, nh, dk), (d[:, nq:nq + nk] + bias[1]).view(T, nkv, dk)
    v = d[:, nq + nk:] + bias[2]
    q, k = P.unit_rms(P.turn_halves(q, pos, rot, 500.0), eps), P.unit_rms(P.turn_halves(k, pos, rot, 500.0), eps)
    inv = torch.tensor([500.0 ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float32, device="cuda")
    out = torch.empty(T, nq, dtype=dtype, device="cuda")
    K.attention_prep(proj.cuda(), 0, nq, nq + nk, nh, nkv, dk, dv, ctx, cache, out, q_bias=bias[0].cuda(), k_bias=bias[1].cuda(),
                     v_bias=bias[2].cuda(), norm_eps=eps, qk_unit=True, inv_freq=inv, rotary_dim=rot)
    tol = 5e-5 if dtype == torch.float32 else 3e-2
    assert (out.double().cpu() - q.reshape(T, -1)).abs().max() < tol
    at = 0
    for r, (ql, kv) in enumerate(zip(q_lens, kv_lens)):
        p = torch.arange(kv - ql, kv)
        page = cache.block_table[r].cpu()[p // 16].long()
        kc, vc = cache.k_pages.cpu()[page, :, p % 16].double(), cache.v_pages.cpu()[page, :, p % 16].double()
        assert (kc - k[at:at + ql]).abs().max() < tol and (vc - v[at:at + ql].reshape(ql, nkv, dv)).abs().max() < tol
        at += ql
    K.check_status()


def _memory_case(q_lens, slots, heads, key_heads, N, V, seed, fixed=False, strong=False):
    """Random operands (bfloat16 numbers in float64), fades from forgetting at once to remembering all, states of
    all slots and what the plain walk makes of them."""
    g = torch.Generator().manual_seed(seed)
    T = sum(q_lens)
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).double()
    q, k, v = bf(T, key_heads, N) / 4, bf(T, key_heads, N) / 4, bf(T, heads, V)
    base = torch.linspace(0.0, 1.0, heads) ** 3 * 0.999 if heads > 1 else torch.tensor([0.01])
    la = -base[None, :] * (0.2 + 2.0 * torch.rand(T, heads, generator=g))
    if strong:
        la = torch.where(torch.rand(T, heads, generator=g) < 0.05, torch.full_like(la, -400.0), la)      # (forgets everything at once)
    write = 0.1 + torch.rand(T, heads, generator=g)
    if fixed:
        la, write = -base[None, :].expand(T, heads).clone(), torch.ones(T, heads)
    la, write = la.float(), write.float()
    start = torch.randn(len(slots) + 2, heads, V, N, generator=g).float()
    out, end, at = torch.zeros(T, heads, V, dtype=F64), start.double().clone(), 0
    for n, slot in zip(q_lens, slots):
        for h in range(heads):
            S = start[slot, h].double().T
            for t in range(at, at + n):
                S = torch.exp(la[t, h].double()) * S + write[t, h].double() * torch.outer(k[t, h // (heads // key_heads)], v[t, h])
                out[t, h] = S.T @ q[t, h // (heads // key_heads)]
            end[slot, h] = S.T
        at += n
    return q, k, v, la, write, start, out.reshape(T, heads * V), end


@pytest.mark.parametrize("q_lens", [[1], [1, 1, 1, 60], [129], [48, 1, 300], [1, 128, 127, 2]])
@pytest.mark.parametrize("heads, key_heads, N, V", [(4, 4, 64, 128), (6, 2, 128, 64), (3, 1, 40, 24), (2, 2, 8, 72), (2, 1, 128, 128), (1, 1, 64, 8)])
@pytest.mark.parametrize("strong", [False, True])
def test_memories_in_chunks_and_walked(q_lens, heads, key_heads, N, V, strong):
    """bfloat16 operands through the chunked form (single tokens in front left to the walk) and through the walk
    alone, against the token-by-token recurrence in float64: as exact as 32-bit either way, also where a head
    forgets everything within a chunk, and only the step's slots change."""
    from llm_singularity_b200 import kernels as K
    slots = [2, 0, 4, 1][:len(q_lens)]
    q, k, v, la, write, start, want, end = _memory_case(q_lens, slots, heads, key_heads, N, V, N + V + len(q_lens), strong=strong)
    T, KH = sum(q_lens), key_heads * N
    ctx = _ctx(q_lens, [n + 5 for n in q_lens], rows=slots)
    rows = torch.cat([q.reshape(T, KH), k.reshape(T, KH), v.reshape(T, heads * V)], dim=1).to(torch.bfloat16).cuda()
    fades = torch.stack([torch.exp(la), write, la]).cuda()
    tol = 3e-5 * float(want.abs().max())
    for chunked in (False, True):
        state, out = start.cuda(), torch.zeros(T, heads * V, device="cuda")
        first = K.chunk_scan_first(ctx, torch.bfloat16, N, V) if chunked else None
        assert (first is not None) == (chunked and max(q_lens) >= 48) and (first is None or first == (3 if q_lens[0] == 1 and len(q_lens) == 4 and q_lens[1] == 1
                                                                                                        else 1 if q_lens == [1, 128, 127, 2] else 0))
        if first != 0:
            K.linear_scan(rows, 0, KH, 2 * KH, heads, N, V, "given", None, None, None, "none", "none", "none", state, ctx, out,
                          keep=fades[0], write=fades[1], key_heads=key_heads, requests=first, q_scale=0.5)
        if first is not None:
            K.chunk_scan(rows, 0, KH, 2 * KH, heads, key_heads, N, V, state, ctx, out, first, log_keep=fades[2], write=fades[1], q_scale=0.5)
        err = (out.double().cpu() - 0.5 * want).abs().max()
        assert err < tol, (chunked, float(err), float(want.abs().max()))
        assert (state.double().cpu() - end).abs().max() < 3e-5 * float(end.abs().max()), chunked
    K.check_status()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("q_lens", [[1, 1], [3, 1, 20], [1, 200, 60]])
@pytest.mark.parametrize("heads, D, V, rot", [(3, 20, 28, 14), (2, 64, 128, 64), (4, 8, 16, 2), (2, 128, 64, 128)])
def test_retention_as_a_part(dtype, q_lens, heads, D, V, rot):
    """Projection, rotation at far positions, memory, unit heads, gate and output of a retention mixer, the state
    carried over two steps."""
    from llm_singularity_b200.config.specs import LinearRecurrenceSpec, RotarySpec
    from llm_singularity_b200.parts import MIXERS, Runtime
    from llm_singularity_b200.parts.base import StateView
    g = torch.Generator().manual_seed(D + V)
    H, base, eps, T = 64, 700.0, 1e-5, sum(q_lens)
    decay = tuple(float(x) for x in torch.linspace(0.5, 1.0, heads))
    shapes = {"q": (heads * D, H), "k": (heads * D, H), "v": (heads * V, H), "g": (heads * V, H), "o": (H, heads * V)}
    W = {n: (torch.randn(s, generator=g) / math.sqrt(s[1])).to(torch.bfloat16) for n, s in shapes.items()}
    rt = Runtime("cuda", dtype)
    part = MIXERS.build(LinearRecurrenceSpec(hidden_size=H, num_heads=heads, key_dim=D, value_dim=V, decay=decay, q_activation="none",
                                             k_activation="none", out_norm="unit", out_gate=True, out_gate_activation="silu", eps=eps,
                                             position=RotarySpec(head_dim=D, rotary_dim=rot, theta=base), k_scale=D ** -0.5), rt)
    part.load({n: t.to("cuda", dtype) for n, t in W.items()})
    state = torch.zeros(4, heads, V, D, device="cuda")
    m = {"heads": heads, "dim": D, "vdim": V, "decay": decay, "rot": {"dims": rot, "base": base}}
    xs = [torch.randn(2 * n, H, generator=g).to(torch.bfloat16) for n in q_lens]
    Wd = {n: t.double() for n, t in W.items()}
    want = [P.retention(x.double(), Wd, "", m, torch.arange(2 * n) + 1000, eps) for x, n in zip(xs, q_lens)]
    slots = [3, 0, 2][:len(q_lens)]
    for half in (0, 1):
        ctx = _ctx(q_lens, [1000 + (1 + half) * n for n in q_lens], rows=slots)
        x = torch.cat([x[half * n:(half + 1) * n] for x, n in zip(xs, q_lens)]).to("cuda", dtype)
        got = part.forward(x, ctx, StateView(state)).double().cpu()
        ref = torch.cat([w[half * n:(half + 1) * n] for w, n in zip(want, q_lens)])
        assert (got - ref).abs().max() < (1e-4 if dtype == torch.float32 else 6e-2) * max(1.0, float(ref.abs().max())), (half, (got - ref).abs().max())


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads, V, G, N, taps, groups", [(4, 16, 2, 8, 4, 2), (3, 7, 1, 5, 3, 7), (2, 64, 2, 64, 2, 1), (5, 4, 1, 12, 1, 5), (2, 24, 1, 16, 6, 3)])
def test_around_the_state_space_walk(dtype, heads, V, G, N, taps, groups):
    """Convolution with its carried inputs (portions shorter than the taps, single tokens alone in a step and
    beside portions), step sizes and fades, skip, gate and group norm, over three steps."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(heads + V)
    inner, gn = heads * V, G * N
    C, cols, eps = inner + 2 * gn, 2 * inner + 2 * gn + heads, 1e-5
    steps = [[3, 1, 20], [1, 1, 1], [2, 70, 1]]
    slots = [2, 0, 3]
    conv, conv_b = torch.randn(C, taps, generator=g) / math.sqrt(taps), torch.randn(C, generator=g)
    dt_b, a_log, D, w = torch.randn(heads, generator=g), torch.randn(heads, generator=g), torch.randn(heads, generator=g), torch.randn(inner, generator=g)
    lens = [sum(s[r] for s in steps) for r in range(3)]
    raw = [torch.randn(n, cols, generator=g) for n in lens]
    for r in raw:
        r[:, -heads:] *= 8.0                                         # (step sizes on both ends of softplus)
    ys = [torch.randn(n, inner, generator=g) for n in lens]
    us = [P.silu(P.short_conv(r.double()[:, inner:inner + C], conv.double(), conv_b.double())) for r in raw]
    state = torch.zeros(4, max(taps - 1, 1), C, device="cuda") if taps > 1 else None
    at = [0, 0, 0]
    tol = 5e-5 if dtype == torch.float32 else 4e-2
    for step in steps:
        cut = lambda xs: torch.cat([x[a:a + n] for x, a, n in zip(xs, at, step)])
        T, rows = sum(step), cut(raw)
        ctx = _ctx(step, [a + n for a, n in zip(at, step)], rows=slots)
        proj = rows.cuda()
        u, fades = torch.empty(T, C, dtype=dtype, device="cuda"), torch.empty(3, T, heads, device="cuda")
        K.state_space_prep(proj, inner, inner + C, C, conv.cuda(), conv_b.cuda(), dt_b.cuda(), a_log.cuda(), state, ctx, u, fades)
        assert (u.double().cpu() - cut(us)).abs().max() < tol * 2
        step_size = P.softplus(rows.double()[:, cols - heads:] + dt_b.double())
        fade = -torch.exp(a_log.double()) * step_size
        for got, ref in zip(fades.double().cpu(), (torch.exp(fade), step_size, fade)):
            assert ((got - ref).abs() <= 2e-6 * (1.0 + ref.abs())).all()
        out = torch.empty(T, inner, dtype=dtype, device="cuda")
        K.state_space_output(cut(ys).cuda(), proj, inner, u, D.repeat_interleave(V).cuda(), w.cuda(), heads, groups, eps, taps, state, ctx, out)
        v = (cut(ys).double().view(T, heads, V) + D.double()[:, None] * u.double().cpu()[:, :inner].view(T, heads, V)).reshape(T, inner)
        v = v * P.silu(rows.double()[:, :inner])
        want = P.unit_rms(v.view(T, groups, inner // groups), eps).reshape(T, inner) * w.double()
        assert ((out.double().cpu() - want).abs() <= tol * (1.0 + want.abs())).all()
        at = [a + n for a, n in zip(at, step)]
    K.check_status()


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("hidden", [52, 128, 2050, 4096, 5000])
def test_norm_behind_a_sublayer_and_the_sum(dtype, hidden):
    """A weighted sum of results with a bias, and the sum over a token's experts, normed and joined to the 32-bit
    stream; the copy is the new stream rounded."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(hidden)
    T, eps, top, cap = 11, 1e-5, 6, 70
    w, bias = torch.randn(hidden, generator=g), torch.randn(hidden, generator=g)
    ys = [torch.randn(T, hidden, generator=g).to(dtype) for _ in range(3)]
    scales = [0.5, -2.0, 3.0]
    rows = torch.randn(cap, hidden, generator=g)
    pos, wts = torch.randperm(cap, generator=g)[:T * top].to(torch.int32), torch.rand(T, top, generator=g)
    cases = [(ys, scales, bias, None), (ys[:1], [1.0], None, None), ([rows.to(dtype)], [1.0], None, pos), ([rows], [1.0], bias, pos)]
    for terms, sc, b, places in cases:
        x = torch.randn(T, hidden, generator=g)
        if places is None:
            v = sum(s * y.double() for s, y in zip(sc, terms))
        else:
            v = (terms[0].double()[pos.long()].view(T, top, hidden) * wts.double()[:, :, None]).sum(1)
        v = v + (b.double() if b is not None else 0.0)
        want = x.double() + P.unit_rms(v, eps) * w.double()
        for copy_dtype in (None, dtype):
            stream = x.cuda()
            copy = None if copy_dtype is None else torch.empty(T, hidden, dtype=dtype, device="cuda")
            K.join_norm(stream, [t.cuda() for t in terms], sc, b.cuda() if b is not None else None, w.cuda(), eps, copy,
                        pos=places.cuda() if places is not None else None, wts=wts.cuda() if places is not None else None)
            assert (stream.double().cpu() - want).abs().max() < 2e-5
            if copy is not None:
                assert torch.equal(copy, stream.to(dtype))
    K.check_status()


def test_bias_of_the_output_projection_without_a_pair(tmp_path):
    """The sum of branches with a bias as a kernel of its own (a caller that does not form it)."""
    from llm_singularity_b200 import kernels as K
    g = torch.Generator().manual_seed(2)
    for dtype in TYPES:
        a, b, bias = torch.randn(5, 70, generator=g).to(dtype), torch.randn(5, 70, generator=g).to(dtype), torch.randn(70, generator=g)
        out = torch.empty(5, 70, dtype=dtype, device="cuda")
        K.branch_sum([a.cuda(), b.cuda()], [2.0, -0.5], out, bias=bias.cuda())
        want = 2.0 * a.double() - 0.5 * b.double() + bias.double()
        assert (out.double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("T, H, F, E, top, vocab", [(5, 64, 48, 6, 2, 30), (300, 64, 48, 6, 3, 11), (33, 52, 18, 4, 4, 50), (1, 128, 64, 9, 1, 7),
                                                    (700, 136, 264, 5, 2, 400), (3, 64, 16, 40, 35, 9)])
def test_experts_named_by_tables(dtype, T, H, F, E, top, vocab):
    """Three layers' tables planned in one launch; every layer's own experts, the sum formed there and left open."""
    from llm_singularity_b200.config.specs import MoESpec
    from llm_singularity_b200.parts import FEED_FORWARDS, Runtime
    g = torch.Generator().manual_seed(T + H)
    rt = Runtime("cuda", dtype)
    toks = torch.randint(0, vocab, (T,), generator=g).tolist()
    toks[0], toks[-1] = vocab - 1, 0
    ctx = _ctx([T], [T], tokens=[toks])
    parts, weights = [], []
    for _ in range(3):
        W = {"table": torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)}
        for e in range(E):
            for n, s in (("gate", (F, H)), ("up", (F, H)), ("down", (H, F))):
                W[f"e{e}.{n}"] = (torch.randn(s, generator=g) / math.sqrt(s[1])).to(torch.bfloat16)
        part = FEED_FORWARDS.build(MoESpec(hidden_size=H, expert_size=F, num_experts=E, top=top, weight_on="output", token_rows=vocab), rt)
        part.load({n: t.cuda() if t.dtype == torch.int32 else t.to("cuda", dtype) for n, t in W.items()})
        parts.append(part)
        weights.append({n: t.double() for n, t in W.items()})
    for i, p in enumerate(parts):
        p.share_plans([q.table for q in parts], i)
    x = torch.randn(T, H, generator=g).to(torch.bfloat16)
    for part, W in zip(parts, weights):
        want = P.experts_by_token(x.double(), W, "", {"router": {"top": top}}, toks)
        got = part.forward(x.to("cuda", dtype), ctx)
        tol = (1e-5 if dtype == torch.float32 else 4e-2) * max(1.0, float(want.abs().max()))
        assert (got.double().cpu() - want).abs().max() < tol
        rows = part.forward(x.to("cuda", dtype), ctx, open_sum=True)
        summed = (rows.rows.double()[rows.places.long()].view(T, top, H) * rows.weights.double()[:, :, None]).sum(1).cpu()
        assert (summed - want).abs().max() < tol
    assert len(ctx.expert_plans) == 1
    rt.ops.check_status()


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
