"""MofidraConfig: the Mofidra decoder's configuration, read from config.json keys.

A Mofidra model is a list of layers of differential attention (two softmax maps per head over one
value, the second taken off the first; rotary positions on each map) with a feed-forward of one of
two kinds or none.  Both sublayers of a layer read the output of one norm and are added to the
stream together.  Feed-forwards: ``dense`` (two products around the tanh form of gelu) or ``moe`` (a
biased router whose weights are the softmax over the chosen logits, ungated experts with the square
of relu, an optional shared expert behind a sigmoid of one number per token).  The norms' stored
weights are distances from one.  A stretch of layers may run several times in a row with the same
weights (``loop``), each pass with caches of its own.  The embedding is scaled on the way in; the
output head has a matrix of its own.  Every size and constant below comes from config.json; the
tensor names are those of the checkpoint.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Mapping, Optional, Tuple

from .llama import ConfigError
from .specs import (DenseMLPSpec, EmbeddingSpec, HeadSpec, KVAttentionSpec, LayerCall, ModelSpec, MoESpec, NoPositionSpec,
                    RMSNormSpec, RotarySpec, SideBySideBlockSpec)

MIXER_KINDS = ("attention",)
MLP_KINDS = ("dense", "moe")
DENSE_ACTIVATION = "gelu_tanh"
EXPERT_ACTIVATION = "relu_squared"


def _get(d: Mapping[str, Any], key: str, where: str):
    if not isinstance(d, Mapping) or key not in d or d[key] is None:
        raise ConfigError(f"config.json: {where} lacks '{key}'")
    return d[key]


def _pos_int(d: Mapping[str, Any], key: str, where: str) -> int:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {where} '{key}' must be a positive integer, got {v!r}")
    return v


def _count(d: Mapping[str, Any], key: str, where: str) -> int:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"config.json: {where} '{key}' must be an integer, not negative, got {v!r}")
    return v


def _number(d: Mapping[str, Any], key: str, where: str) -> float:
    v = _get(d, key, where)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where} '{key}' must be a number, got {v!r}")
    return float(v)


def _pos_float(d: Mapping[str, Any], key: str, where: str) -> float:
    v = _number(d, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where} '{key}' must be positive, got {v!r}")
    return v


@dataclass(frozen=True)
class MofidraAttention:
    heads: int
    kv_heads: int
    dim: int                          # of one map's query and key
    vdim: int
    scale: float
    diff: float                       # the constant part of the second map's factor
    rot_dims: int = 0                 # 0: no rotation
    rot_base: float = 10000.0


@dataclass(frozen=True)
class MofidraMLP:
    kind: str
    ff: int                           # dense: hidden size; moe: an expert's
    experts: int = 0
    top: int = 0
    shared_ff: int = 0                # 0: no shared expert


@dataclass(frozen=True)
class MofidraLayer:
    mixer: MofidraAttention
    mlp: Optional[MofidraMLP] = None


@dataclass(frozen=True)
class MofidraConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[MofidraLayer, ...]
    loop_start: int = 0               # layers loop_start .. loop_stop - 1 run loop_times times in a row
    loop_stop: int = 0
    loop_times: int = 0               # 0: no loop

    architecture = "Mofidra"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MofidraConfig":
        norm = _get(d, "norm", "the model")
        raw_layers = _get(d, "layers", "the model")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = tuple(cls._parse_layer(i, e) for i, e in enumerate(raw_layers))
        kw = {}
        loop = d.get("loop")
        if loop:
            kw = dict(loop_start=_count(loop, "start", "'loop'"), loop_stop=_count(loop, "stop", "'loop'"),
                      loop_times=_pos_int(loop, "times", "'loop'"))
        emb = d.get("embedding") or {}
        cfg = cls(vocab=_pos_int(d, "vocab", "the model"), width=_pos_int(d, "width", "the model"),
                  norm_eps=_pos_float(norm, "eps", "'norm'"),
                  embedding_scale=_number(emb, "scale", "'embedding'") if emb.get("scale") is not None else 1.0,
                  layers=layers, **kw)
        cfg.validate()
        return cfg

    @staticmethod
    def _parse_mixer(m: Mapping[str, Any], where: str) -> MofidraAttention:
        heads = _pos_int(m, "heads", where)
        kw = dict(heads=heads, kv_heads=_pos_int(m, "kv_heads", where) if m.get("kv_heads") is not None else heads,
                  dim=_pos_int(m, "dim", where), vdim=_pos_int(m, "vdim", where), scale=_number(m, "scale", where),
                  diff=_number(m, "diff", where))
        rot = m.get("rot")
        if rot:
            kw.update(rot_dims=_pos_int(rot, "dims", where + " rot"), rot_base=_pos_float(rot, "base", where + " rot"))
        return MofidraAttention(**kw)

    @staticmethod
    def _parse_mlp(mlp: Mapping[str, Any], where: str) -> MofidraMLP:
        kind = mlp.get("kind", "dense")
        if kind not in MLP_KINDS:
            raise ConfigError(f"config.json: {where} has a feed-forward of kind '{kind}' (known: {', '.join(MLP_KINDS)})")
        if kind == "dense":
            return MofidraMLP("dense", ff=_pos_int(mlp, "ff", where + " mlp"))
        expert, router = _get(mlp, "expert", where + " mlp"), _get(mlp, "router", where + " mlp")
        shared = mlp.get("shared")
        return MofidraMLP("moe", ff=_pos_int(expert, "ff", where + " expert"),
                          experts=_pos_int(router, "experts", where + " router"), top=_pos_int(router, "top", where + " router"),
                          shared_ff=_pos_int(shared, "ff", where + " shared") if shared else 0)

    @classmethod
    def _parse_layer(cls, i: int, entry: Mapping[str, Any]) -> MofidraLayer:
        where = f"layer {i}"
        kind = _get(entry, "type", where)
        if kind not in MIXER_KINDS:
            raise ConfigError(f"config.json: {where} has type '{kind}' (known: {', '.join(MIXER_KINDS)})")
        mlp = entry.get("mlp")
        return MofidraLayer(cls._parse_mixer(_get(entry, "mixer", where), where),
                            None if mlp is None else cls._parse_mlp(mlp, where))

    def validate(self) -> None:
        if self.loop_times and not 0 <= self.loop_start < self.loop_stop <= len(self.layers):
            raise ConfigError(f"loop: layers {self.loop_start} .. {self.loop_stop} - 1 of {len(self.layers)}")
        for i, l in enumerate(self.layers):
            m = l.mixer
            if m.heads % m.kv_heads:
                raise ConfigError(f"layer {i}: {m.heads} heads cannot share {m.kv_heads} kv heads")
            if m.rot_dims % 2 or m.rot_dims > m.dim:
                raise ConfigError(f"layer {i}: rot.dims {m.rot_dims} must be even and at most dim {m.dim}")
            if l.mlp is not None and l.mlp.kind == "moe" and l.mlp.top > l.mlp.experts:
                raise ConfigError(f"layer {i}: top {l.mlp.top} of {l.mlp.experts} experts")

    # ------------------------------------------------------------------ writing
    @staticmethod
    def _mixer_dict(m: MofidraAttention) -> dict:
        d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "diff": m.diff}
        if m.rot_dims:
            d["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
        return d

    @staticmethod
    def _mlp_dict(f: Optional[MofidraMLP]):
        if f is None:
            return None
        if f.kind == "dense":
            return {"kind": "dense", "ff": f.ff}
        d = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
        if f.shared_ff:
            d["shared"] = {"ff": f.shared_ff}
        return d

    def to_dict(self) -> dict:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "embedding": {"scale": self.embedding_scale},
             "layers": [{"type": "attention", "mixer": self._mixer_dict(l.mixer), "mlp": self._mlp_dict(l.mlp)}
                        for l in self.layers]}
        if self.loop_times:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        return d

    # -------------------------------------------------------------- translation
    def run_order(self) -> List[int]:
        """The layers' numbers in the order they run."""
        n = len(self.layers)
        if not self.loop_times:
            return list(range(n))
        a, b = self.loop_start, self.loop_stop
        return list(range(a)) + list(range(a, b)) * self.loop_times + list(range(b, n))

    def _mixer_spec(self, m: MofidraAttention) -> KVAttentionSpec:
        position = NoPositionSpec()
        if m.rot_dims:
            position = RotarySpec(head_dim=m.dim, rotary_dim=m.rot_dims, theta=m.rot_base, pairing="half")
        return KVAttentionSpec(hidden_size=self.width, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim,
                               value_dim=m.vdim, scale=m.scale, eps=self.norm_eps, position=position, diff=m.diff)

    def _ffn_spec(self, f: Optional[MofidraMLP]):
        if f is None:
            return None
        W = self.width
        if f.kind == "dense":
            return DenseMLPSpec(hidden_size=W, intermediate_size=f.ff, activation=DENSE_ACTIVATION)
        shared = None
        if f.shared_ff:
            shared = DenseMLPSpec(hidden_size=W, intermediate_size=f.shared_ff, activation=EXPERT_ACTIVATION)
        return MoESpec(hidden_size=W, expert_size=f.ff, num_experts=f.experts, top=f.top, activation=EXPERT_ACTIVATION,
                       score="softmax_chosen", weight_on="output", gated=False, router_bias=True, shared=shared,
                       shared_gate=shared is not None)

    @staticmethod
    def _mlp_names(f: MofidraMLP, p: str, b: str):
        """(checkpoint name, (owner path, the part's parameter)) of a layer's feed-forward."""
        if f.kind == "dense":
            return [(p + "up", (b, "up_proj")), (p + "down", (b, "down_proj"))]
        names = [(p + "router", (b, "router")), (p + "router.b", (b, "router_bias"))]
        for e in range(f.experts):
            names += [(f"{p}e{e}.{w}", (b, f"e{e}.{w}")) for w in ("up", "down")]
        if f.shared_ff:
            names += [(f"{p}shared.{w}", (b + ".shared", w + "_proj")) for w in ("up", "down")]
            names.append((p + "shared.sg", (b, "shared_gate")))
        return names

    def to_model_spec(self) -> ModelSpec:
        W = self.width
        norm = RMSNormSpec(size=W, eps=self.norm_eps, unit_offset=True)
        names = [("embed", ("embedding", "weight")), ("final.norm", ("head.norm", "weight")), ("head", ("head", "weight"))]
        blocks = []
        for i, l in enumerate(self.layers):
            p, b = f"l{i}.", f"blocks.{i}"
            blocks.append(SideBySideBlockSpec(mixer=self._mixer_spec(l.mixer), ffn=self._ffn_spec(l.mlp), norm=norm))
            names.append((p + "norm1", (b + ".norm", "weight")))
            names += [(f"{p}mix.{n}", (b + ".mixer", n)) for n in ("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2")]
            if l.mlp is not None:
                names += self._mlp_names(l.mlp, p + "mlp.", b + ".ffn")
        # every run of a layer has a cache of its own: a pass through looped layers shares weights only
        order = tuple(LayerCall(block=i, cache=c) for c, i in enumerate(self.run_order()))
        return ModelSpec(
            architecture=self.architecture,
            embedding=EmbeddingSpec(vocab_size=self.vocab, hidden_size=W, scale=self.embedding_scale),
            blocks=tuple(blocks), order=order,
            head=HeadSpec(vocab_size=self.vocab, hidden_size=W, tied=False, norm=norm),
            tensor_names=tuple(names))
