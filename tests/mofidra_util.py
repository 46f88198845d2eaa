"""Small Mofidra models for the tests: configurations that differ in every size, random weights made
here (not by the engine), and helpers that step the engine and compare with tests/plain_mofidra.py.

The sizes are chosen so that nothing passes by two sizes being equal or a count being one: key and
value sizes differ, kv heads are one, several or as many as the heads, heads are rotated wholly, in part
or not at all, experts are chosen one, two or three at a time with and without a shared expert,
layers come with and without feed-forward, the loop covers a part of the layers or is left out, and the
constant of the second map differs from layer to layer.
"""
import json
import math
import os

import torch

import plain_mofidra
from zinizen_util import close, make_runner, position_errors, rel_err, run_cuts, tokens_for  # noqa: F401  (any design)


def att(heads, kv, dim, vdim, diff, rot=None, scale=None):
    """``rot``: (rotated dims, base) or None."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale or 1.0 / math.sqrt(dim)}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def model(width, vocab, layers, eps=1e-5, scale=None, loop=None):
    """``layers``: (mixer, feed-forward) pairs; ``loop``: (start, stop, times)."""
    cfg = {"architecture": "Mofidra", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "embedding": {"scale": 1.0 if scale is None else scale},
           "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


CONFIGS = {
    # nothing a multiple of eight; the loop in the middle, three times round
    "mix_a": model(72, 211, [
        (att(6, 3, 20, 12, 0.2, rot=(20, 300.0)), moe(5, 2, 22, shared=34)),
        (att(4, 1, 10, 36, 0.7, rot=(6, 1000.0), scale=0.45), dense(50)),
        (att(3, 3, 14, 18, 0.35), None),
        (att(9, 3, 12, 10, 0.5, rot=(4, 77.0)), moe(7, 3, 18)),
    ], eps=2e-5, scale=3.0, loop=(1, 3, 3)),
    # sizes that fill whole tiles (the tensor-core paths in bfloat16); the loop from the first layer on
    "mix_b": model(128, 160, [
        (att(4, 2, 64, 128, 0.3, rot=(64, 50000.0)), moe(8, 2, 64, shared=96)),
        (att(8, 2, 32, 64, 0.6, rot=(16, 10000.0)), dense(192)),
        (att(2, 2, 128, 128, 0.8, rot=(128, 1e6)), moe(16, 4, 32)),
        (att(6, 1, 24, 40, 0.45, rot=(24, 500.0)), moe(6, 1, 48, shared=64)),
    ], eps=1e-6, scale=11.0, loop=(0, 2, 2)),
    # counts that are one, sizes that are equal, no loop, no scale
    "mix_c": model(48, 53, [
        (att(1, 1, 16, 16, 0.5, rot=(16, 50.0)), moe(3, 1, 48)),
        (att(2, 2, 8, 8, 0.1, rot=(2, 10.0)), moe(2, 2, 8, shared=8)),
        (att(3, 1, 16, 256, 0.9), None),
    ]),
}


def single(mlp="dense", **kw):
    """A one-layer model."""
    mixer = att(kw.get("heads", 6), kw.get("kv", 2), kw.get("dim", 24), kw.get("vdim", 40), kw.get("diff", 0.4),
                kw.get("rot", (16, 1000.0)), kw.get("scale"))
    ff = {"dense": dense(44), "moe": moe(kw.get("experts", 6), kw.get("top", 2), 20, shared=kw.get("shared", 28)), None: None}[mlp]
    return model(56, 97, [(mixer, ff)], scale=kw.get("emb", 2.0), loop=kw.get("loop"))


def typed(cfg):
    from llm_singularity_b200.config.mofidra import MofidraConfig
    return MofidraConfig.from_dict(cfg)


def make_weights(cfg, seed, sharpen=2.0):
    """Random bfloat16-representable weights, name -> float32 tensor.  Queries and keys are scaled up so that
    the softmax is peaked and one wrong or missing key shows; routers are scaled up and their biases are
    as large as the logits, so that the bias changes choices and weights; the four vectors of the second
    map's factor move it well away from its constant part.  In a model of several layers the routed
    feed-forwards speak softly, so that what a router's close call changes under bfloat16 rounding stays
    within rounding (in 32-bit nothing flips, and one-layer models keep the full weight)."""
    from llm_singularity_b200.engine.runner import expected_tensors_of
    g = torch.Generator().manual_seed(seed)
    soft = 0.2 if len(cfg["layers"]) > 1 else 1.0
    out = {}
    for name, (shape, role, init) in expected_tensors_of(typed(cfg).to_model_spec()).items():
        n = torch.randn(shape, generator=g)
        if name.endswith("norm1") or name == "final.norm":
            t = 0.2 * n
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            # (products of about 0.3 and -0.2)
            t = (1.0 + 0.3 * n) * math.sqrt((0.3 if name.endswith("1") else 0.2) / shape[0]) * (-1.0 if name.endswith("lk2") else 1.0)
        elif name.endswith("router.b"):
            t = 1.5 * n
        elif name == "embed":
            t = n
        else:
            t = n / math.sqrt(shape[1])
            if name.endswith((".mix.q", ".mix.k")):
                t = t * sharpen
            elif name.endswith(".router"):
                t = t * 3.0
            elif name.endswith(".sg"):
                t = t * 2.0
            elif ".mlp.e" in name and name.endswith(".down"):
                t = t * soft
        out[name] = t.to(torch.bfloat16).float()
    return out


def write_model(path, cfg, weights, dtype=torch.bfloat16):
    from llm_singularity_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"), {n: t.to(dtype) for n, t in weights.items()})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return path


def plain_logits(cfg, weights, tokens):
    return plain_mofidra.forward(cfg, weights, tokens).float()
