"""Typed configuration of the Vaderax design, read from config.json.

The file lists the layers one by one: each entry names its mixer (`type`), the mixer's sizes and constants (`mixer`)
and its feed-forward (`mlp`, or null).  Nothing is assumed about their order, and no size or constant has a stand-in
in code: what a layer needs and the file lacks is an error that names the key.

    architecture     "Vaderax"
    vocab, width     vocabulary and residual width
    norm.eps         eps of every norm
    embedding.scale  the constant every embedded row is multiplied by
    layers[i].type   "delta" | "attention"
    layers[i].mixer  delta:     heads, kv_heads (query/key heads), dim, vdim, conv (taps)
                     attention: heads, kv_heads, dim, vdim, scale, rot.base, rot.dims
    layers[i].mlp    null; kind "dense" with ff; kind "moe" with expert.ff and router.{experts, top} and optionally
                     router.identity (outputs of the router that stand for the input itself) and
                     router.groups.{count, keep}
    loop             may be absent; start, stop, times: layers start .. stop - 1 run `times` times in a row, every pass
                     with a cache of its own, and before every pass but the first the embedding output is added to x

A layer is x <- x + mixer(norm1(x)), then x <- x + mlp(norm2(x)), the norms layer norms with weight and bias.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .bepuzen import MAX_POSITIONS, _need, _pos_float, _pos_int
from .funevik import _rot
from .qwen3 import ConfigError
from .spec import LayerRun, LayerSpec, ModelSpec, PartSpec
from .torisun import _count
from .vifelix import _number


@dataclass(frozen=True)
class DeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float
    rot_dims: int


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                   # "dense" | "moe"
    ff: int                     # dense: its size; moe: the size of one expert
    experts: int = 0
    top: int = 0
    identity: int = 0           # router outputs behind the experts' that stand for the input itself
    groups: int = 1             # the experts and identity experts form this many equal groups of neighbours
    keep: int = 1               # groups that a token may choose from


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


MixerConfig = Union[DeltaConfig, AttentionConfig]


@dataclass(frozen=True)
class VaderaxConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embedding_scale: float
    mixers: Tuple[MixerConfig, ...]
    mlps: Tuple[Optional[FeedForwardConfig], ...]
    loop: Optional[LoopConfig] = None
    eos_token_id: Optional[int] = None
    torch_dtype: str = "bfloat16"

    ARCHITECTURE = "Vaderax"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "VaderaxConfig":
        layers = _need(d, "layers", "")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config key 'layers' must be a non-empty list")
        eps = _pos_float(_need(d, "norm", ""), "eps", "norm.")
        mixers, mlps = [], []
        for i, L in enumerate(layers):
            at = f"layers[{i}]."
            kind = _need(L, "type", at)
            m = _need(L, "mixer", at)
            if kind == "delta":
                mixers.append(cls._delta(m, at + "mixer."))
            elif kind == "attention":
                mixers.append(cls._attention(m, at + "mixer."))
            else:
                raise ConfigError(f"{at}type={kind!r} is not a mixer of this design (delta, attention)")
            mlps.append(cls._mlp(L.get("mlp"), at + "mlp."))
        eos = d.get("eos_token_id")
        return cls(architecture=cls.ARCHITECTURE, vocab_size=_pos_int(d, "vocab", ""), hidden_size=_pos_int(d, "width", ""),
                   norm_eps=eps, embedding_scale=_number(_need(d, "embedding", ""), "scale", "embedding."),
                   mixers=tuple(mixers), mlps=tuple(mlps), loop=cls._loop(d.get("loop"), len(layers)),
                   eos_token_id=eos if isinstance(eos, int) else None, torch_dtype=str(d.get("torch_dtype", "bfloat16")))

    @staticmethod
    def _heads(m: Mapping[str, Any], at: str) -> Dict[str, int]:
        s = {k: _pos_int(m, k, at) for k in ("heads", "kv_heads", "dim", "vdim")}
        if s["heads"] % s["kv_heads"]:
            raise ConfigError(f"{at}heads={s['heads']} must be a multiple of kv_heads={s['kv_heads']}")
        return s

    @classmethod
    def _delta(cls, m: Mapping[str, Any], at: str) -> DeltaConfig:
        return DeltaConfig(taps=_pos_int(m, "conv", at), **cls._heads(m, at))

    @classmethod
    def _attention(cls, m: Mapping[str, Any], at: str) -> AttentionConfig:
        s = cls._heads(m, at)
        base, dims = _rot(m, at, s["dim"])
        return AttentionConfig(scale=_pos_float(m, "scale", at), rot_base=base, rot_dims=dims, **s)

    @staticmethod
    def _mlp(mlp: Optional[Mapping[str, Any]], at: str) -> Optional[FeedForwardConfig]:
        if mlp is None:
            return None
        kind = _need(mlp, "kind", at)
        if kind == "dense":
            return FeedForwardConfig("dense", _pos_int(mlp, "ff", at))
        if kind == "moe":
            router, rt = _need(mlp, "router", at), at + "router."
            g = router.get("groups")
            c = FeedForwardConfig("moe", _pos_int(_need(mlp, "expert", at), "ff", at + "expert."), experts=_pos_int(router, "experts", rt),
                                  top=_pos_int(router, "top", rt),
                                  identity=_count(router, "identity", rt) if router.get("identity") is not None else 0,
                                  groups=_pos_int(g, "count", rt + "groups.") if g is not None else 1,
                                  keep=_pos_int(g, "keep", rt + "groups.") if g is not None else 1)
            choices = c.experts + c.identity
            if choices % c.groups:
                raise ConfigError(f"{rt}groups.count={c.groups} must divide the {choices} experts and identity experts")
            if c.keep > c.groups:
                raise ConfigError(f"{rt}groups.keep={c.keep} exceeds groups.count={c.groups}")
            if c.top > choices // c.groups * c.keep:
                raise ConfigError(f"{rt}top={c.top} exceeds the {choices // c.groups * c.keep} experts of the groups kept")
            return c
        raise ConfigError(f"{at}kind={kind!r} is not a feed-forward of this design (dense, moe)")

    @staticmethod
    def _loop(loop: Optional[Mapping[str, Any]], layers: int) -> Optional[LoopConfig]:
        if loop is None:
            return None
        c = LoopConfig(_count(loop, "start", "loop."), _count(loop, "stop", "loop."), _pos_int(loop, "times", "loop."))
        if not c.start <= c.stop <= layers:
            raise ConfigError(f"loop.start={c.start} .. loop.stop={c.stop} is not a range of the {layers} layers")
        return c

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for m, f in zip(self.mixers, self.mlps):
            mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
            if isinstance(m, DeltaConfig):
                kind = "delta"
                mixer["conv"] = m.taps
            else:
                kind = "attention"
                mixer.update({"scale": m.scale, "rot": {"base": m.rot_base, "dims": m.rot_dims}})
            mlp: Optional[Dict[str, Any]] = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top, "identity": f.identity,
                                                                         "groups": {"count": f.groups, "keep": f.keep}}}
            layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "layers": layers}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    # ------------------------------------------------------------------ the model as parts
    @property
    def num_hidden_layers(self) -> int:
        return len(self.mixers)

    def order(self) -> Tuple[LayerRun, ...]:
        n = len(self.mixers)
        if self.loop is None:
            return tuple(LayerRun(i) for i in range(n))
        a, b = self.loop.start, self.loop.stop
        body = [LayerRun(i, add_embedding=again > 0 and i == a) for again in range(self.loop.times) for i in range(a, b)]
        return tuple([LayerRun(i) for i in range(a)] + body + [LayerRun(i) for i in range(b, n)])

    def model_spec(self) -> ModelSpec:
        D, eps = self.hidden_size, self.norm_eps
        norm = PartSpec("layernorm", {"size": D, "eps": eps, "leaf": "", "bias_leaf": "b"})
        block = PartSpec("prenorm_residual", {"mixer_name": "mix", "feed_forward_name": "mlp", "mixer_norm_name": "norm1",
                                              "feed_forward_norm_name": "norm2"})
        layers = []
        for i, (m, f) in enumerate(zip(self.mixers, self.mlps)):
            if isinstance(m, DeltaConfig):
                mixer = PartSpec("gated_delta", {"hidden_size": D, "num_heads": m.heads, "num_qk_heads": m.kv_heads, "qk_dim": m.dim,
                                                 "v_dim": m.vdim, "taps": m.taps, "norm_eps": eps})
            else:
                mixer = PartSpec("gqa_window_sink", {
                    "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "qk_dim": m.dim, "v_dim": m.vdim,
                    "scale": m.scale, "unit_norm_eps": eps, "gate": "sigmoid",
                    "position_encoding": PartSpec("rotary_partial", {"dims": m.rot_dims, "base": m.rot_base})})
            parts = {"mixer": mixer, "mixer_norm": norm}
            if f is not None:
                parts["feed_forward_norm"] = norm
                if f.kind == "dense":
                    parts["feed_forward"] = PartSpec("dense", {"hidden_size": D, "intermediate_size": f.ff, "activation": "relu2"})
                else:
                    parts["feed_forward"] = PartSpec("routed_experts", {
                        "hidden_size": D, "num_experts": f.experts, "top_k": f.top, "expert_size": f.ff, "routing": "softmax",
                        "activation": "relu2", "correction": True, "identity": f.identity, "groups": (f.groups, f.keep)})
            layers.append(LayerSpec(prefix=f"l{i}", block=block, parts=parts))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=D, vocab_size=self.vocab_size, max_positions=MAX_POSITIONS,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab_size, "hidden_size": D, "leaf": "",
                                                   "scale": self.embedding_scale}),
            layers=tuple(layers), order=self.order(), final_norm=norm,
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab_size, "hidden_size": D, "leaf": ""}),
            embedding_prefix="embed", final_norm_prefix="final.norm", lm_head_prefix="head")
        spec.validate()
        return spec

    @staticmethod
    def canonical_tensor_name(name: str) -> str:
        return name

    def ignorable_tensor(self, name: str) -> bool:
        """The norm stored for a feed-forward that the layer does not have."""
        return any(f is None and name in (f"l{i}.norm2", f"l{i}.norm2.b") for i, f in enumerate(self.mlps))
