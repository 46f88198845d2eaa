"""Small Lilupel models for the tests: configurations that differ in every size, random weights made
here (not by the engine), and helpers that step the engine and compare with tests/plain_lilupel.py.

The sizes are chosen so that nothing passes by two sizes being equal or a count being one: key and
value sizes differ, kv heads are one, several or as many as the heads, heads rotate wholly or in part and
the two mixers of a pair rotate differently, windows are shorter than a page in one model and span
several pages in another, convolutions have one to five taps, state-space memories have one, some or as many
groups as heads and norm groups that do not fall on heads, tokens have one to four experts, layers come
with and without feed-forward and borrow weights from layers of either kind.
"""
import json
import math
import os

import torch

import plain_lilupel
from zinizen_util import TOLERANCE, make_runner, position_errors, rel_err, run_cuts, tokens_for  # noqa: F401  (any design)


def close(got, want, dtype):
    """32-bit: every position within the tolerance.  bfloat16: a retention head's output is brought to unit rms
    whatever its size, so where its first tokens' products nearly cancel, rounding turns the head round, and the
    positions behind it remember that; so one position in seven (and always one) may be outside, and the median must lie
    well inside.  A fault of the cache, the state or the batch shows in 32-bit, where no such allowance is made."""
    e = position_errors(got, want)
    if dtype == "float32":
        return bool(e.max() < TOLERANCE[dtype])
    return bool((e > TOLERANCE[dtype]).sum() <= max(1, len(e) // 7) and e.median() < TOLERANCE[dtype] / 2)


def att(heads, kv, dim, vdim, window, rot, scale=None):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 2.5 / math.sqrt(dim),
            "mask": {"size": window}, "rot": {"dims": rot[0], "base": rot[1]}}


def ret(heads, dim, vdim, rot, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot[0], "base": rot[1]},
            "decay": decay or [1.0 - 2.0 ** (-2.0 - 5.0 * h / heads) for h in range(heads)]}


def pair(left, right, left_scale=0.7, right_scale=1.3):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def space(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp, of=None):
    e = {"type": "parallel" if "left" in mixer else "mamba2", "mixer": mixer, "mlp": mlp}
    if of is not None:
        e["weights_of"] = of
    return e


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Lilupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


_A0 = pair(att(6, 3, 20, 12, 24, (8, 5000.0)), ret(3, 18, 10, (14, 300.0)))
_A1 = space(6, 10, 12, 3, 3, 5)
_B0 = pair(att(4, 2, 64, 64, 40, (64, 10000.0)), ret(2, 64, 128, (64, 100000.0)), 1.2, -0.4)
_B1 = space(4, 64, 128, 2, 4, 2)
_B2 = pair(att(4, 1, 32, 48, 33, (16, 1000.0)), ret(4, 24, 72, (16, 50.0)))
_C0 = pair(att(1, 1, 16, 16, 5, (16, 50.0)), ret(1, 16, 16, (2, 10.0)), 1.0, 1.0)

CONFIGS = {
    # nothing a multiple of eight, both kinds borrowed
    "mix_a": model(76, 211, [
        layer(_A0, moe(7, 2, 22)),
        layer(_A1, None),
        layer(pair(att(5, 1, 10, 14, 70, (10, 77.0)), ret(5, 6, 22, (6, 1e4)), 0.3, 1.0), moe(5, 4, 18)),
        layer(_A1, None, of=1),
        layer(space(3, 14, 6, 1, 5, 1), moe(7, 2, 22)),
        layer(_A0, moe(7, 2, 22), of=0),
    ], eps=3e-5),
    # sizes that fill whole tiles (the tensor-core paths in bfloat16)
    "mix_b": model(128, 160, [
        layer(_B1, moe(8, 2, 64)),
        layer(_B0, moe(8, 2, 64)),
        layer(_B1, moe(8, 2, 64), of=0),
        layer(_B2, moe(12, 3, 40)),
        layer(space(6, 24, 40, 6, 2, 3), None),
    ], eps=1e-6),
    # counts that are one, sizes that are equal, windows shorter than a page, no convolution
    "mix_c": model(48, 53, [
        layer(_C0, moe(3, 1, 48)),
        layer(space(1, 16, 16, 1, 1, 1), moe(2, 2, 8)),
        layer(_C0, moe(3, 1, 48), of=0),
    ]),
}


def single(kind, mlp=True, **kw):
    """A one-layer model of one mixer kind."""
    if kind == "parallel":
        mixer = pair(att(kw.get("heads", 6), kw.get("kv", 2), kw.get("dim", 24), kw.get("vdim", 40), kw.get("window", 50),
                         kw.get("rot", (12, 2000.0)), kw.get("scale")),
                     ret(kw.get("rheads", 3), kw.get("rdim", 20), kw.get("rvdim", 28), kw.get("rrot", (20, 700.0)), kw.get("decay")),
                     kw.get("left_scale", 0.6), kw.get("right_scale", 0.9))
    else:
        mixer = space(kw.get("heads", 6), kw.get("vdim", 20), kw.get("state", 12), kw.get("groups", 2), kw.get("conv", 4),
                      kw.get("norm_groups", 3))
    return model(56, 97, [layer(mixer, moe(kw.get("experts", 6), kw.get("top", 2), 20) if mlp else None)])


def typed(cfg):
    from llm_singularity_b200.config.lilupel import LilupelConfig
    return LilupelConfig.from_dict(cfg)


def make_weights(cfg, seed):
    """Random bfloat16-representable weights, name -> float32 tensor (tables of experts int32, rows of different
    numbers).  Sinks are as large as the scores; step sizes and fades of the state-space memories run from heads
    that forget in a token to heads that remember hundreds."""
    from llm_singularity_b200.engine.runner import expected_tensors_of
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, (shape, role, init) in expected_tensors_of(typed(cfg).to_model_spec()).items():
        if role == "int_table":
            n = int(init.split(":")[1])
            out[name] = torch.stack([torch.randperm(n, generator=g)[:shape[1]] for _ in range(shape[0])]).to(torch.int32)
            continue
        n = torch.randn(shape, generator=g)
        if name.endswith((".norm1", ".norm2")) or name == "final.norm":
            t = 0.2 * n
        elif name.endswith(".mix.norm"):
            t = 1.0 + 0.2 * n
        elif name.endswith(".sink"):
            t = 1.0 + 1.5 * n
        elif name.endswith(".A_log"):
            t = torch.linspace(-4.0, 1.5, shape[0]) if shape[0] > 1 else torch.zeros(1)
        elif name.endswith(".dt_bias"):
            t = -1.0 + n
        elif name.endswith(".D"):
            t = 1.0 + 0.5 * n
        elif name.endswith(".conv"):
            t = n / math.sqrt(shape[1])
        elif name.endswith(".b"):
            t = 0.3 * n
        elif name == "embed":
            t = n
        else:
            t = n / math.sqrt(shape[1])
        out[name] = t.to(torch.bfloat16).float()
    return out


def write_model(path, cfg, weights, dtype=torch.bfloat16):
    from llm_singularity_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {n: t if t.dtype == torch.int32 else t.to(dtype) for n, t in weights.items()})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return path


def plain_logits(cfg, weights, tokens):
    return plain_lilupel.forward(cfg, weights, tokens).float()
