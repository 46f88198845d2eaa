"""The Lilupel design on the host: its configuration (reading, refusals, writing back), the model spec it
becomes (parts, tensor names, run order, what every layer keeps per request), tables of experts in the
random-weights mode, and properties of the plain model that the GPU tests rely on."""
import copy
import math

import pytest
import torch

import lilupel_util as U
import plain_lilupel as P
from llm_singularity_b200.config.lilupel import LilupelConfig
from llm_singularity_b200.config.llama import ConfigError
from llm_singularity_b200.config.specs import KVAttentionSpec, LinearRecurrenceSpec, MoESpec, NoPositionSpec, RotarySpec, StateSpaceSpec
from llm_singularity_b200.engine.runner import expected_tensors_of
from llm_singularity_b200.models.decoder import DecoderModel
from llm_singularity_b200.parts import FEED_FORWARDS, MIXERS, CompositeCacheSpec, PagedKVSpec, Runtime, StateSpec
from llm_singularity_b200.registry import architecture_of, load_config

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_configuration_reads_and_writes_back(name, tmp_path):
    cfg = U.CONFIGS[name]
    assert architecture_of(cfg).config_cls is LilupelConfig
    typed = LilupelConfig.from_dict(cfg)
    assert typed.to_dict() == cfg and LilupelConfig.from_dict(typed.to_dict()) == typed
    U.write_model(str(tmp_path), cfg, U.make_weights(cfg, 1))
    assert load_config(str(tmp_path)) == typed


def test_what_may_be_left_out():
    cfg = copy.deepcopy(U.CONFIGS["mix_c"])
    cfg["layers"][0]["mixer"]["left"].pop("kv_heads")
    cfg["layers"][2]["mixer"] = copy.deepcopy(cfg["layers"][0]["mixer"])
    cfg["layers"][1].pop("mlp")
    typed = LilupelConfig.from_dict(cfg)
    assert typed.layers[0].left.kv_heads == 1 and typed.layers[1].mlp is None


def test_refusals_name_the_layer():
    cases = [(lambda c: c["layers"][0].update(type="conv"), "layer 0"),
             (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "layer 0"),
             (lambda c: c["layers"][2]["mixer"]["left"]["rot"].update(dims=12), "layer 2"),
             (lambda c: c["layers"][2]["mixer"]["right"]["rot"].update(dims=5), "layer 2"),
             (lambda c: c["layers"][2]["mixer"]["right"].update(decay=[0.5]), "layer 2"),
             (lambda c: c["layers"][2]["mixer"]["right"].update(decay="slow"), "layer 2"),
             (lambda c: c["layers"][2]["mixer"]["left"].pop("mask"), "layer 2"),
             (lambda c: c["layers"][2]["mixer"].pop("right_scale"), "layer 2"),
             (lambda c: c["layers"][4]["mixer"].update(groups=2), "layer 4"),
             (lambda c: c["layers"][4]["mixer"].update(norm_groups=4), "layer 4"),
             (lambda c: c["layers"][4]["mixer"].update(conv=0), "layer 4"),
             (lambda c: c["layers"][4]["mlp"]["router"].update(top=8), "layer 4"),
             (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "layer 0"),
             (lambda c: c["layers"][5].update(weights_of=6), "layer 5"),
             (lambda c: c["layers"][5].update(weights_of=5), "layer 5"),
             (lambda c: c["layers"][5].update(weights_of=1), "layer 5"),
             (lambda c: c["norm"].pop("eps"), "norm"),
             (lambda c: c.pop("vocab"), "vocab")]
    for change, where in cases:
        cfg = copy.deepcopy(U.CONFIGS["mix_a"])
        change(cfg)
        with pytest.raises(ConfigError) as e:
            LilupelConfig.from_dict(cfg)
        assert where in str(e.value)


def test_spec_parts_names_order_and_caches():
    spec = LilupelConfig.from_dict(U.CONFIGS["mix_a"]).to_model_spec()
    assert [b.kind for b in spec.blocks] == ["output_norm"] * 4
    assert [(c.block, c.cache) for c in spec.order] == [(0, 0), (1, 1), (2, 2), (1, 3), (3, 4), (0, 5)]
    left, right = spec.blocks[0].mixer.branches
    assert left.sink and left.sink_logit and left.qk_unit and left.qkv_bias and left.out_bias and left.window == 24
    assert left.position.rotary_dim == 8 and right.position.rotary_dim == 14 and right.k_scale == pytest.approx(18 ** -0.5)
    assert right.out_norm == "unit" and right.out_gate_activation == "silu" and spec.blocks[0].mixer.scales == (0.7, 1.3)
    assert spec.blocks[1].ffn is None and spec.blocks[0].ffn.token_rows == 211 and spec.blocks[0].mixer_norm.unit_offset
    assert spec.head.tied and spec.head.norm.unit_offset
    names = expected_tensors_of(spec)
    assert names["l0.mix.left.q.b"][0] == (120,) and names["l0.mix.left.o"][0] == (76, 72) and names["l0.mix.left.o.b"][0] == (76,)
    assert names["l0.mix.left.sink"][0] == (6,) and names["l0.mix.right.g"][0] == (30, 76) and "l0.mix.right.norm" not in names
    assert names["l1.mix.in"][0] == (2 * 60 + 2 * 36 + 6, 76) and names["l1.mix.conv"][0] == (132, 3) and names["l1.mix.norm"][0] == (60,)
    assert names["l0.mlp.table"] == ((211, 2), "int_table", "distinct:7") and names["l2.mlp.e4.down"][0] == (76, 18)
    assert "l1.norm2" not in names and "l5.norm1" not in names and "head" not in names and "l0.mlp.router" not in names
    model = DecoderModel(spec, Runtime("cpu", torch.float32, ops=object()))
    caches = model.cache_specs()
    assert isinstance(caches[0], CompositeCacheSpec) and caches[0].paged and caches[0].window == 24 and not caches[0].shareable
    assert caches[0].parts == (PagedKVSpec(3, 20, 24, 12), StateSpec((3, 10, 18))) and caches[5] == caches[0]
    assert caches[1].parts == (StateSpec((6, 10, 12)), StateSpec((2, 132))) and caches[3] == caches[1]
    plain = DecoderModel(LilupelConfig.from_dict(U.CONFIGS["mix_c"]).to_model_spec(), Runtime("cpu", torch.float32, ops=object()))
    assert plain.cache_specs()[1].parts == (StateSpec((1, 16, 16)),)          # one tap: no inputs to keep


def test_weights_may_be_borrowed_through_a_borrower():
    cfg = copy.deepcopy(U.CONFIGS["mix_c"])
    cfg["layers"].append(copy.deepcopy(cfg["layers"][2]))
    cfg["layers"][3]["weights_of"] = 2
    typed = LilupelConfig.from_dict(cfg)
    assert typed.weight_layer(3) == 0 and [c.block for c in typed.to_model_spec().order] == [0, 1, 0, 0]


def test_parts_refuse_what_they_do_not_combine():
    rt = Runtime("cpu", torch.float32, ops=object())
    att = dict(hidden_size=32, num_heads=2, num_kv_heads=1, key_dim=16, value_dim=16, scale=0.25)
    for bad in (dict(sink_logit=True), dict(qk_unit=True, qk_norm=True), dict(diff=0.5, out_bias=True)):
        with pytest.raises(ValueError):
            MIXERS.build(KVAttentionSpec(**att, **bad), rt)
    rec = dict(hidden_size=32, num_heads=2, key_dim=8, value_dim=8, decay=(0.5, 0.9))
    turn = RotarySpec(head_dim=8, rotary_dim=8)
    MIXERS.build(LinearRecurrenceSpec(**rec, q_activation="none", k_activation="none", position=turn), rt)
    for bad in (dict(position=turn), dict(out_norm="some"), dict(out_gate_activation="tanh"), dict(gate="forget", k_scale=0.5),
                dict(q_activation="none", k_activation="none", position=RotarySpec(head_dim=8, rotary_dim=8, pairing="adjacent"))):
        with pytest.raises(ValueError):
            MIXERS.build(LinearRecurrenceSpec(**{**rec, **bad}), rt)
    for bad in (dict(groups=4), dict(norm_groups=5), dict(conv_taps=0)):
        with pytest.raises(ValueError):
            MIXERS.build(StateSpaceSpec(**{**dict(hidden_size=32, num_heads=6, groups=2, state_dim=8, value_dim=4), **bad}), rt)
    for bad in (dict(weight_on="input"), dict(router_bias=True), dict(choice_bias=True)):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build(MoESpec(**{**dict(hidden_size=32, expert_size=8, num_experts=4, top=2, token_rows=10,
                                                  weight_on="output"), **bad}), rt)
    assert isinstance(MIXERS.build(LinearRecurrenceSpec(**rec), rt).spec.position, NoPositionSpec)


def test_tables_of_experts_are_checked_and_made_at_random():
    from llm_singularity_b200.weights.random_init import random_tensors
    cfg = U.CONFIGS["mix_a"]
    spec = LilupelConfig.from_dict(cfg).to_model_spec()
    made = random_tensors(expected_tensors_of(spec), 5)
    for name, n, top in (("l0.mlp.table", 7, 2), ("l2.mlp.table", 5, 4)):
        t = made[name]
        assert t.dtype == torch.int32 and tuple(t.shape) == (211, top) and 0 <= int(t.min()) and int(t.max()) < n
        assert all(len(set(r)) == top for r in t.tolist()) and len({tuple(r) for r in t.tolist()}) > n
    assert torch.equal(made["l0.mlp.table"], random_tensors(expected_tensors_of(spec), 5)["l0.mlp.table"])
    model = DecoderModel(spec, Runtime("cpu", torch.float32, ops=object()))
    model.load_tensors({n: t.float() if t.dtype != torch.int32 else t for n, t in made.items()})
    ffns = [b.ffn for b in model.blocks if b.ffn is not None]
    assert len(ffns[0].tables) == 2 and ffns[0].tables[1] is ffns[2].table and ffns[2].index == 1 and len(ffns[1].tables) == 1
    made["l2.mlp.table"][3, 1] = 5
    with pytest.raises(ValueError, match="experts"):
        model.load_tensors({n: t.float() if t.dtype != torch.int32 else t for n, t in made.items()})


# ------------------------------------------------------------------ the plain model itself
def test_sink_takes_weight_and_is_not_scaled():
    s = torch.tensor([[0.5, 9.0], [1.0, -2.0]], dtype=F64)
    ok = torch.tensor([[True, False], [True, True]])
    w = P.softmax_beside_sink(s, torch.tensor(1.0, dtype=F64), ok)
    assert w[0].tolist() == pytest.approx([math.exp(0.5) / (math.exp(0.5) + math.e), 0.0])
    assert w[1].tolist() == pytest.approx([math.e / (2 * math.e + math.exp(-2)), math.exp(-2) / (2 * math.e + math.exp(-2))])
    assert float(P.softmax_beside_sink(s, torch.tensor(900.0, dtype=F64), ok).sum()) == 0.0


def test_norm_before_or_after_the_rotation_is_the_same():
    g = torch.Generator().manual_seed(3)
    v, pos = torch.randn(9, 2, 10, generator=g, dtype=F64), torch.arange(9) * 1000
    assert torch.allclose(P.unit_rms(P.turn_halves(v, pos, 6, 300.0), 1e-5), P.turn_halves(P.unit_rms(v, 1e-5), pos, 6, 300.0))


def test_memory_is_a_sum_over_the_past():
    g = torch.Generator().manual_seed(4)
    q, k, v = (torch.randn(7, n, generator=g, dtype=F64) for n in (3, 3, 2))
    keep, write = torch.rand(7, generator=g, dtype=F64), torch.rand(7, generator=g, dtype=F64)
    got = P.fading_memory(q, k, v, keep, write)
    for t in range(7):
        want = sum(write[s] * torch.prod(keep[s + 1:t + 1]) * (q[t] @ k[s]) * v[s] for s in range(t + 1))
        assert torch.allclose(got[t], want)


def test_every_mechanism_matters():
    """Changing any tensor of the model changes the logits by far more than the tests' tolerances."""
    for kind in ("parallel", "mamba2"):
        cfg = U.single(kind)
        W = U.make_weights(cfg, 5)
        toks = U.tokens_for(cfg, 60, 1)
        base = P.forward(cfg, W, toks)
        for name in W:
            other = dict(W)
            if name.endswith("table"):
                other[name] = (W[name] + 1) % 6
            elif ".mlp.e" in name and name.split(".")[2] != "e1":
                continue
            else:
                other[name] = W[name] + 0.5 * W[name].abs().mean() * torch.randn(W[name].shape, generator=torch.Generator().manual_seed(9))
            assert U.rel_err(P.forward(cfg, other, toks), base) > 0.004, name


def test_borrowed_weights_are_the_layer_written_out():
    cfg = U.CONFIGS["mix_a"]
    W = U.make_weights(cfg, 3)
    toks = U.tokens_for(cfg, 12, 2)
    flat, W2 = copy.deepcopy(cfg), dict(W)
    for i, l in enumerate(flat["layers"]):
        j = l.pop("weights_of", i)
        if j != i:
            W2.update({f"l{i}." + n.split(".", 1)[1]: t for n, t in W.items() if n.startswith(f"l{j}.")})
    assert torch.equal(P.forward(cfg, W, toks), P.forward(flat, W2, toks))
