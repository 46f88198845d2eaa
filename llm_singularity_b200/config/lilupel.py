"""LilupelConfig: the Lilupel decoder's configuration, read from config.json keys.

A Lilupel model is a list of layers whose two sublayers read the residual stream itself, with a norm
behind each (``x += norm1(mixer(x))``, then ``x += norm2(ff(x))`` where the layer has a feed-forward).
Mixers: ``parallel``, windowed attention with biased projections, normed and rotated heads and a learnt
sink per head beside a retention memory (a fixed decay per head, rotated queries and keys, a gated
output), added with fixed factors; or ``mamba2``, a state-space memory behind a short convolution.
The feed-forward is a set of gated experts without a router: a table names the experts of every token
id.  The norms' stored weights are distances from one.  A layer may use another layer's weights
(``weights_of``) with a cache or state of its own.  The embedding table is also the output head.  Every
size and constant below comes from config.json; the tensor names are those of the checkpoint.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .llama import ConfigError
from .mofidra import _get, _number, _pos_float, _pos_int
from .specs import (EmbeddingSpec, HeadSpec, KVAttentionSpec, LayerCall, LinearRecurrenceSpec, ModelSpec, MoESpec,
                    OutputNormBlockSpec, ParallelMixerSpec, RMSNormSpec, RotarySpec, StateSpaceSpec)

MIXER_KINDS = ("parallel", "mamba2")
EXPERT_ACTIVATION = "silu"


@dataclass(frozen=True)
class LilupelRotation:
    dims: int
    base: float


@dataclass(frozen=True)
class LilupelAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot: LilupelRotation


@dataclass(frozen=True)
class LilupelRetention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: LilupelRotation


@dataclass(frozen=True)
class LilupelStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class LilupelExperts:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class LilupelLayer:
    kind: str
    left: Optional[LilupelAttention] = None
    right: Optional[LilupelRetention] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    space: Optional[LilupelStateSpace] = None             # the ``mamba2`` mixer
    mlp: Optional[LilupelExperts] = None                  # None: no feed-forward
    weights_of: Optional[int] = None                      # the layer whose tensors this one uses

    def description(self):
        """What a layer that borrows this one's weights must share with it."""
        return (self.kind, self.left, self.right, self.left_scale, self.right_scale, self.space, self.mlp)


@dataclass(frozen=True)
class LilupelConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[LilupelLayer, ...]

    architecture = "Lilupel"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LilupelConfig":
        norm = _get(d, "norm", "the model")
        raw_layers = _get(d, "layers", "the model")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        cfg = cls(vocab=_pos_int(d, "vocab", "the model"), width=_pos_int(d, "width", "the model"),
                  norm_eps=_pos_float(norm, "eps", "'norm'"),
                  layers=tuple(cls._parse_layer(i, e) for i, e in enumerate(raw_layers)))
        cfg.validate()
        return cfg

    @staticmethod
    def _parse_rot(m: Mapping[str, Any], where: str) -> LilupelRotation:
        rot = _get(m, "rot", where)
        return LilupelRotation(_pos_int(rot, "dims", where + " rot"), _pos_float(rot, "base", where + " rot"))

    @classmethod
    def _parse_left(cls, m: Mapping[str, Any], where: str) -> LilupelAttention:
        heads = _pos_int(m, "heads", where)
        return LilupelAttention(
            heads=heads, kv_heads=_pos_int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads,
            dim=_pos_int(m, "dim", where), vdim=_pos_int(m, "vdim", where), scale=_pos_float(m, "scale", where),
            window=_pos_int(_get(m, "mask", where), "size", where + " mask"), rot=cls._parse_rot(m, where))

    @classmethod
    def _parse_right(cls, m: Mapping[str, Any], where: str) -> LilupelRetention:
        decay = _get(m, "decay", where)
        if not isinstance(decay, (list, tuple)) or not all(isinstance(x, (int, float)) and not isinstance(x, bool) for x in decay):
            raise ConfigError(f"config.json: {where} 'decay' must be a list of numbers, got {decay!r}")
        return LilupelRetention(heads=_pos_int(m, "heads", where), dim=_pos_int(m, "dim", where), vdim=_pos_int(m, "vdim", where),
                                decay=tuple(float(x) for x in decay), rot=cls._parse_rot(m, where))

    @staticmethod
    def _parse_space(m: Mapping[str, Any], where: str) -> LilupelStateSpace:
        return LilupelStateSpace(**{k: _pos_int(m, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})

    @staticmethod
    def _parse_mlp(mlp: Mapping[str, Any], where: str) -> LilupelExperts:
        if mlp.get("kind", "moe") != "moe":
            raise ConfigError(f"config.json: {where} has a feed-forward of kind '{mlp.get('kind')}' (known: moe)")
        expert, router = _get(mlp, "expert", where + " mlp"), _get(mlp, "router", where + " mlp")
        return LilupelExperts(ff=_pos_int(expert, "ff", where + " expert"), experts=_pos_int(router, "experts", where + " router"),
                              top=_pos_int(router, "top", where + " router"))

    @classmethod
    def _parse_layer(cls, i: int, entry: Mapping[str, Any]) -> LilupelLayer:
        where = f"layer {i}"
        kind = _get(entry, "type", where)
        if kind not in MIXER_KINDS:
            raise ConfigError(f"config.json: {where} has type '{kind}' (known: {', '.join(MIXER_KINDS)})")
        m = _get(entry, "mixer", where)
        of = entry.get("weights_of")
        if of is not None and (isinstance(of, bool) or not isinstance(of, int)):
            raise ConfigError(f"config.json: {where} 'weights_of' must name a layer by its number, got {of!r}")
        mlp = entry.get("mlp")
        kw = dict(mlp=None if mlp is None else cls._parse_mlp(mlp, where), weights_of=of)
        if kind == "mamba2":
            return LilupelLayer(kind, space=cls._parse_space(m, where), **kw)
        return LilupelLayer(kind, left=cls._parse_left(_get(m, "left", where), where + " left"),
                            right=cls._parse_right(_get(m, "right", where), where + " right"),
                            left_scale=_number(m, "left_scale", where), right_scale=_number(m, "right_scale", where), **kw)

    def validate(self) -> None:
        for i, l in enumerate(self.layers):
            for side, m in (("left", l.left), ("right", l.right)):
                if m is not None and (m.rot.dims % 2 or m.rot.dims > m.dim):
                    raise ConfigError(f"layer {i} {side}: rot.dims {m.rot.dims} must be even and at most dim {m.dim}")
            if l.left is not None and l.left.heads % l.left.kv_heads:
                raise ConfigError(f"layer {i}: {l.left.heads} heads cannot share {l.left.kv_heads} kv heads")
            if l.right is not None and len(l.right.decay) != l.right.heads:
                raise ConfigError(f"layer {i}: {len(l.right.decay)} decays for {l.right.heads} heads")
            s = l.space
            if s is not None:
                if s.heads % s.groups:
                    raise ConfigError(f"layer {i}: {s.heads} heads cannot share {s.groups} groups")
                if s.heads * s.vdim % s.norm_groups:
                    raise ConfigError(f"layer {i}: {s.norm_groups} norm groups do not divide {s.heads} heads of {s.vdim}")
            if l.mlp is not None and l.mlp.top > l.mlp.experts:
                raise ConfigError(f"layer {i}: top {l.mlp.top} of {l.mlp.experts} experts")
            if l.weights_of is not None:
                j = self.weight_layer(i)
                if self.layers[j].description() != l.description():
                    raise ConfigError(f"layer {i}: uses the weights of layer {j} but is described differently")

    def weight_layer(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = [i]
        while self.layers[seen[-1]].weights_of is not None:
            j = self.layers[seen[-1]].weights_of
            if not 0 <= j < len(self.layers) or j in seen:
                raise ConfigError(f"layer {i}: weights_of {j} must lead to a layer that has weights of its own")
            seen.append(j)
        return seen[-1]

    # ------------------------------------------------------------------ writing
    @staticmethod
    def _mixer_dict(l: LilupelLayer) -> dict:
        if l.kind == "mamba2":
            s = l.space
            return {"heads": s.heads, "vdim": s.vdim, "state": s.state, "groups": s.groups, "conv": s.conv,
                    "norm_groups": s.norm_groups}
        a, r = l.left, l.right
        rot = lambda m: {"base": m.rot.base, "dims": m.rot.dims}
        return {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                         "mask": {"size": a.window}, "rot": rot(a)},
                "right": {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "decay": list(r.decay), "rot": rot(r)},
                "left_scale": l.left_scale, "right_scale": l.right_scale}

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            f = l.mlp
            e = {"type": l.kind, "mixer": self._mixer_dict(l),
                 "mlp": None if f is None else {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            layers.append(e)
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": layers}

    # -------------------------------------------------------------- translation
    def _mixer_spec(self, l: LilupelLayer):
        W, eps = self.width, self.norm_eps
        turn = lambda m: RotarySpec(head_dim=m.dim, rotary_dim=m.rot.dims, theta=m.rot.base, pairing="half")
        if l.kind == "mamba2":
            s = l.space
            return StateSpaceSpec(hidden_size=W, num_heads=s.heads, groups=s.groups, state_dim=s.state, value_dim=s.vdim,
                                  conv_taps=s.conv, norm_groups=s.norm_groups, eps=eps)
        a, r = l.left, l.right
        left = KVAttentionSpec(hidden_size=W, num_heads=a.heads, num_kv_heads=a.kv_heads, key_dim=a.dim, value_dim=a.vdim,
                               scale=a.scale, window=a.window, qkv_bias=True, qk_unit=True, eps=eps, sink=True, sink_logit=True,
                               out_bias=True, position=turn(a))
        right = LinearRecurrenceSpec(hidden_size=W, num_heads=r.heads, key_dim=r.dim, value_dim=r.vdim, gate="fixed_decay",
                                     decay=r.decay, q_activation="none", k_activation="none", out_norm="unit", out_gate=True,
                                     out_gate_activation="silu", eps=eps, position=turn(r), k_scale=r.dim ** -0.5)
        return ParallelMixerSpec(hidden_size=W, branches=(left, right), names=("left", "right"), combine="weighted_sum",
                                 scales=(l.left_scale, l.right_scale), eps=eps)

    @staticmethod
    def _mixer_names(l: LilupelLayer, p: str, b: str):
        """(checkpoint name, (owner path, the part's parameter)) of a layer's mixer."""
        if l.kind == "mamba2":
            pairs = [("in", "in"), ("conv", "conv"), ("conv.b", "conv_bias"), ("dt_bias", "dt_bias"), ("A_log", "A_log"),
                     ("D", "D"), ("norm", "norm"), ("o", "o")]
            return [(p + ck, (b, local)) for ck, local in pairs]
        left = [("q", "q"), ("q.b", "q_bias"), ("k", "k"), ("k.b", "k_bias"), ("v", "v"), ("v.b", "v_bias"), ("sink", "sink"),
                ("o", "o"), ("o.b", "o_bias")]
        return ([(p + "left." + ck, (b + ".left", local)) for ck, local in left] +
                [(p + "right." + n, (b + ".right", n)) for n in ("q", "k", "v", "g", "o")])

    def to_model_spec(self) -> ModelSpec:
        W = self.width
        norm = RMSNormSpec(size=W, eps=self.norm_eps, unit_offset=True)
        names = [("embed", ("embedding", "weight")), ("final.norm", ("head.norm", "weight"))]
        blocks, block_of = [], {}
        for i, l in enumerate(self.layers):
            if l.weights_of is not None:
                continue
            p, b, f = f"l{i}.", f"blocks.{len(blocks)}", l.mlp
            block_of[i] = len(blocks)
            ffn = None
            if f is not None:
                ffn = MoESpec(hidden_size=W, expert_size=f.ff, num_experts=f.experts, top=f.top, activation=EXPERT_ACTIVATION,
                              weight_on="output", token_rows=self.vocab)
            blocks.append(OutputNormBlockSpec(mixer=self._mixer_spec(l), ffn=ffn, mixer_norm=norm,
                                              ffn_norm=norm if ffn is not None else None))
            names.append((p + "norm1", (b + ".mixer_norm", "weight")))
            names += self._mixer_names(l, p + "mix.", b + ".mixer")
            if ffn is not None:
                names += [(p + "norm2", (b + ".ffn_norm", "weight")), (p + "mlp.table", (b + ".ffn", "table"))]
                names += [(f"{p}mlp.e{e}.{w}", (b + ".ffn", f"e{e}.{w}")) for e in range(f.experts) for w in ("gate", "up", "down")]
        # every layer has a cache of its own, also one that borrows its weights
        order = tuple(LayerCall(block=block_of[self.weight_layer(i)], cache=i) for i in range(len(self.layers)))
        return ModelSpec(
            architecture=self.architecture,
            embedding=EmbeddingSpec(vocab_size=self.vocab, hidden_size=W),
            blocks=tuple(blocks), order=order,
            head=HeadSpec(vocab_size=self.vocab, hidden_size=W, tied=True, norm=norm),
            tensor_names=tuple(names))
