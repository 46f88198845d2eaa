"""The Mofidra design on the host: its configuration (reading, refusals, writing back), the model spec
it becomes (parts, tensor names, run order, what every layer run keeps per request), and properties of
the plain model that the GPU tests rely on."""
import copy

import pytest
import torch

import mofidra_util as U
import plain_mofidra as P
from llm_singularity_b200.config.llama import ConfigError
from llm_singularity_b200.config.mofidra import MofidraConfig
from llm_singularity_b200.config.specs import KVAttentionSpec, MoESpec
from llm_singularity_b200.engine.runner import expected_tensors_of
from llm_singularity_b200.models.decoder import DecoderModel
from llm_singularity_b200.parts import MIXERS, FEED_FORWARDS, PagedKVSpec, Runtime
from llm_singularity_b200.registry import architecture_of

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_configuration_reads_and_writes_back(name):
    cfg = U.CONFIGS[name]
    assert architecture_of(cfg).config_cls is MofidraConfig
    typed = MofidraConfig.from_dict(cfg)
    assert typed.to_dict() == cfg
    assert MofidraConfig.from_dict(typed.to_dict()) == typed


def test_what_may_be_left_out():
    cfg = copy.deepcopy(U.CONFIGS["mix_c"])
    cfg.pop("embedding")
    cfg["loop"] = None
    cfg["layers"][0]["mixer"].pop("kv_heads")
    cfg["layers"][1]["mlp"]["shared"] = None
    cfg["layers"][2].pop("mlp")
    typed = MofidraConfig.from_dict(cfg)
    assert typed.embedding_scale == 1.0 and typed.run_order() == [0, 1, 2]
    assert typed.layers[0].mixer.kv_heads == 1 and typed.layers[1].mlp.shared_ff == 0 and typed.layers[2].mlp is None


def test_refusals_name_the_layer():
    base = U.CONFIGS["mix_a"]
    cases = [(lambda c: c["layers"][0].update(type="conv"), "layer 0"),
             (lambda c: c["layers"][3]["mixer"].update(kv_heads=2), "layer 3"),
             (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=22), "layer 0"),
             (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "layer 1"),
             (lambda c: c["layers"][2]["mixer"].pop("diff"), "layer 2"),
             (lambda c: c["layers"][2]["mixer"].update(vdim=0), "layer 2"),
             (lambda c: c["layers"][3]["mlp"]["router"].update(top=9), "layer 3"),
             (lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "layer 0"),
             (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "layer 0"),
             (lambda c: c["loop"].update(stop=5), "loop"),
             (lambda c: c["loop"].update(start=3), "loop"),
             (lambda c: c["norm"].pop("eps"), "norm"),
             (lambda c: c.pop("width"), "width")]
    for change, where in cases:
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(ConfigError) as e:
            MofidraConfig.from_dict(cfg)
        assert where in str(e.value)


def test_spec_parts_names_order_and_caches():
    cfg = U.CONFIGS["mix_a"]
    spec = MofidraConfig.from_dict(cfg).to_model_spec()
    assert [b.kind for b in spec.blocks] == ["side_by_side"] * 4
    assert [b.mixer.kind for b in spec.blocks] == ["kv_attention"] * 4
    assert [b.mixer.diff for b in spec.blocks] == [0.2, 0.7, 0.35, 0.5]
    assert [b.mixer.position.kind for b in spec.blocks] == ["rotary", "rotary", "none", "rotary"]
    assert spec.blocks[2].ffn is None and spec.blocks[1].ffn.activation == "gelu_tanh"
    ffn = spec.blocks[0].ffn
    assert (ffn.kind, ffn.score, ffn.weight_on, ffn.gated, ffn.router_bias, ffn.activation) == \
        ("moe", "softmax_chosen", "output", False, True, "relu_squared")
    assert ffn.shared.intermediate_size == 34 and ffn.shared_gate
    assert spec.blocks[3].ffn.shared is None and not spec.blocks[3].ffn.shared_gate
    # every run of a layer has a cache of its own
    assert [(c.block, c.cache) for c in spec.order] == [(0, 0), (1, 1), (2, 2), (1, 3), (2, 4), (1, 5), (2, 6), (3, 7)]
    names = expected_tensors_of(spec)
    assert names["l0.mix.q"][0] == (6 * 2 * 20, 72) and names["l0.mix.k"][0] == (3 * 2 * 20, 72) and names["l0.mix.v"][0] == (36, 72)
    assert names["l1.mix.lq2"][0] == (10,) and names["l1.mix.o"][0] == (72, 144)
    assert names["l0.mlp.router.b"][0] == (5,) and names["l0.mlp.shared.sg"][0] == (1, 72) and names["l0.mlp.e4.down"][0] == (72, 22)
    assert "l3.mlp.shared.sg" not in names and "l0.mlp.e0.gate" not in names and "l0.norm2" not in names
    assert names["head"][0] == (211, 72) and not spec.head.tied and spec.embedding.scale == 3.0
    model = DecoderModel(spec, Runtime("cpu", torch.float32, ops=object()))
    caches = model.cache_specs()
    assert len(caches) == 8
    assert caches[0] == PagedKVSpec(3, 40, None, 12) and caches[1] == caches[3] == caches[5] == PagedKVSpec(1, 20, None, 36)


def test_parts_refuse_what_they_do_not_combine():
    rt = Runtime("cpu", torch.float32, ops=object())
    base = dict(hidden_size=32, num_heads=2, num_kv_heads=1, key_dim=16, value_dim=16, scale=0.25, diff=0.5)
    MIXERS.build(KVAttentionSpec(**base, window=8, chunk=16), rt)
    for extra in (dict(sink=True), dict(qk_norm=True), dict(out_gate=True), dict(logit_softcap=3.0), dict(linear_bias=True)):
        with pytest.raises(ValueError):
            MIXERS.build(KVAttentionSpec(**base, **extra), rt)
    for extra in (dict(shared_gate=True), dict(router_bias=True, choice_bias=True), dict(score="softmax_some")):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(MoESpec(hidden_size=32, expert_size=8, num_experts=4, top=2, **extra), rt)


# ------------------------------------------------------------------ the plain model itself
def test_softmax_over_the_chosen_is_not_over_all():
    z = torch.tensor([[1.0, 3.0, 2.0, -1.0]], dtype=F64)
    ids, w = P.choose(z, 2)
    assert ids.tolist() == [[1, 2]] and torch.allclose(w, torch.softmax(torch.tensor([[3.0, 2.0]], dtype=F64), -1))
    assert not torch.allclose(w, torch.softmax(z, -1)[:, ids[0]])


def test_second_map_and_its_factor_matter():
    cfg = U.single(None)
    W = U.make_weights(cfg, 5)
    toks = U.tokens_for(cfg, 40, 1)
    base = P.forward(cfg, W, toks)
    lam = P.map_mixing({n: t.to(F64) for n, t in W.items()}, "l0.mix.", cfg["layers"][0]["mixer"]["diff"])
    assert abs(lam - cfg["layers"][0]["mixer"]["diff"]) > 0.02
    for n in ("l0.mix.lq1", "l0.mix.lk2"):
        other = dict(W, **{n: -W[n]})
        assert U.rel_err(P.forward(cfg, other, toks), base) > 0.02, n
    q = W["l0.mix.q"].clone().view(6, 2, 24, 56)
    swapped = dict(W, **{"l0.mix.q": q.flip(1).reshape(288, 56)})
    assert U.rel_err(P.forward(cfg, swapped, toks), base) > 0.1


def test_rotation_pairs_halves_of_each_map():
    v = torch.zeros(2, 1, 2, 6, dtype=F64)
    v[1, 0, 0, 0] = v[1, 0, 1, 1] = 1.0
    out = P.turn_halves(v, torch.tensor([0, 1]), 4, 100.0)
    assert torch.allclose(out[1, 0, 0, [0, 2]], torch.tensor([1.0, 1.0], dtype=F64) * torch.tensor([0.5403023059, 0.8414709848], dtype=F64))
    assert torch.allclose(out[1, 0, 1, [1, 3]], torch.tensor([0.9950041653, 0.0998334166], dtype=F64))
    assert torch.equal(out[..., 4:], v[..., 4:]) and torch.equal(out[0], v[0])


def test_a_looped_stretch_is_the_layers_written_out():
    cfg = U.CONFIGS["mix_b"]
    W = U.make_weights(cfg, 3)
    toks = U.tokens_for(cfg, 12, 2)
    flat, W2 = copy.deepcopy(cfg), {}
    flat.pop("loop")
    flat["layers"] = [cfg["layers"][i] for i in P.run_order(cfg)]
    for j, i in enumerate(P.run_order(cfg)):
        W2.update({f"l{j}." + n.split(".", 1)[1]: t for n, t in W.items() if n.startswith(f"l{i}.")})
    W2.update({n: W[n] for n in ("embed", "final.norm", "head")})
    assert torch.equal(P.forward(cfg, W, toks), P.forward(flat, W2, toks))
