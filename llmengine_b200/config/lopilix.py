"""Typed configuration of the Lopilix design, read from config.json.

The file lists the layers one by one: each entry names its mixer (`type`), the mixer's sizes and constants (`mixer`)
and its feed-forward (`mlp`, or null).  Nothing is assumed about their order, and no size or constant has a stand-in
in code: what a layer needs and the file lacks is an error that names the key.

    architecture     "Lopilix"
    vocab, width     vocabulary and width of a stream
    streams          copies of the residual stream (hyper-connections)
    max_positions    rows of the learned position table, the longest sequence
    norm.eps         eps of every norm
    residual_mult    what a sublayer's result is multiplied by on its way into the streams
    logit_scale      what the logits are multiplied by
    layers[i].type   "attention" | "hgrn2" | "latent_attention"
    layers[i].mixer  attention:        heads, kv_heads, dim (per map), vdim, scale, diff, rot.base, rot.dims
                     hgrn2:            heads, dim, vdim
                     latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot.base, rot.dims
                     (rot.scaling {factor, original, fast, slow} may be absent)
    layers[i].mlp    null; kind "dense" with ff; kind "moe" with expert.ff and router.{experts, top, scale} and optionally
                     router.groups.{count, keep}
    loop             may be absent; start, stop, times: layers start .. stop - 1 run `times` times in a row, every pass
                     with a cache or state of its own

Every sublayer reads a weighted sum of the streams through an RMS norm; its result, times a sigmoid gate made from the
same normed input, goes back into all streams, which are mixed with one another on the way.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .bepuzen import _need, _pos_float, _pos_int
from .funevik import _rot
from .qwen3 import ConfigError
from .spec import LayerRun, LayerSpec, ModelSpec, PartSpec
from .torisun import RotaryScaling
from .vaderax import LoopConfig, VaderaxConfig
from .vifelix import _number


@dataclass(frozen=True)
class RotaryConfig:
    base: float
    dims: int
    scaling: Optional[RotaryScaling] = None

    @staticmethod
    def read(m: Mapping[str, Any], at: str, most: int) -> "RotaryConfig":
        base, dims = _rot(m, at, most)
        sc, w = m["rot"].get("scaling"), at + "rot.scaling."
        return RotaryConfig(base, dims, None if sc is None else RotaryScaling(*(_pos_float(sc, k, w) for k in ("factor", "original", "fast", "slow"))))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(vars(self.scaling))
        return d

    def part(self, interleaved: bool) -> PartSpec:
        return PartSpec("rotary_partial", {"dims": self.dims, "base": self.base, "interleaved": interleaved,
                                           "scaling": None if self.scaling is None else dict(vars(self.scaling))})


@dataclass(frozen=True)
class DifferenceAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                    # query/key size per head and map
    vdim: int
    scale: float
    diff: float
    rot: RotaryConfig

    KIND = "attention"


@dataclass(frozen=True)
class MemoryConfig:
    heads: int
    dim: int
    vdim: int

    KIND = "hgrn2"


@dataclass(frozen=True)
class LatentConfig:
    heads: int
    dim: int                    # unrotated query/key size per head
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: RotaryConfig

    KIND = "latent_attention"


@dataclass(frozen=True)
class FeedForwardConfig:
    kind: str                   # "dense" | "moe"
    ff: int                     # dense: its size; moe: the size of one expert
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    groups: int = 1             # the experts form this many equal groups of neighbours
    keep: int = 1               # groups that a token may choose from


MixerConfig = Union[DifferenceAttentionConfig, MemoryConfig, LatentConfig]


@dataclass(frozen=True)
class LopilixConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    streams: int
    max_positions: int
    norm_eps: float
    residual_mult: float
    logit_scale: float
    mixers: Tuple[MixerConfig, ...]
    mlps: Tuple[Optional[FeedForwardConfig], ...]
    loop: Optional[LoopConfig] = None
    eos_token_id: Optional[int] = None
    torch_dtype: str = "bfloat16"

    ARCHITECTURE = "Lopilix"

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LopilixConfig":
        layers = _need(d, "layers", "")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config key 'layers' must be a non-empty list")
        eps = _pos_float(_need(d, "norm", ""), "eps", "norm.")
        readers = {"attention": cls._attention, "hgrn2": cls._memory, "latent_attention": cls._latent}
        mixers, mlps = [], []
        for i, L in enumerate(layers):
            at = f"layers[{i}]."
            kind = _need(L, "type", at)
            m = _need(L, "mixer", at)
            if kind not in readers:
                raise ConfigError(f"{at}type={kind!r} is not a mixer of this design ({', '.join(readers)})")
            mixers.append(readers[kind](m, at + "mixer."))
            mlps.append(cls._mlp(L.get("mlp"), at + "mlp."))
        eos = d.get("eos_token_id")
        return cls(architecture=cls.ARCHITECTURE, vocab_size=_pos_int(d, "vocab", ""), hidden_size=_pos_int(d, "width", ""),
                   streams=_pos_int(d, "streams", ""), max_positions=_pos_int(d, "max_positions", ""), norm_eps=eps,
                   residual_mult=_number(d, "residual_mult", ""), logit_scale=_number(d, "logit_scale", ""), mixers=tuple(mixers),
                   mlps=tuple(mlps), loop=VaderaxConfig._loop(d.get("loop"), len(layers)),
                   eos_token_id=eos if isinstance(eos, int) else None, torch_dtype=str(d.get("torch_dtype", "bfloat16")))

    @staticmethod
    def _attention(m: Mapping[str, Any], at: str) -> DifferenceAttentionConfig:
        s = {k: _pos_int(m, k, at) for k in ("heads", "kv_heads", "dim", "vdim")}
        if s["heads"] % s["kv_heads"]:
            raise ConfigError(f"{at}heads={s['heads']} must be a multiple of kv_heads={s['kv_heads']}")
        return DifferenceAttentionConfig(scale=_pos_float(m, "scale", at), diff=_number(m, "diff", at), rot=RotaryConfig.read(m, at, s["dim"]), **s)

    @staticmethod
    def _memory(m: Mapping[str, Any], at: str) -> MemoryConfig:
        return MemoryConfig(**{k: _pos_int(m, k, at) for k in ("heads", "dim", "vdim")})

    @staticmethod
    def _latent(m: Mapping[str, Any], at: str) -> LatentConfig:
        s = {k: _pos_int(m, k, at) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}
        return LatentConfig(scale=_pos_float(m, "scale", at), rot=RotaryConfig.read(m, at, s["rot_dim"]), **s)

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
                                  top=_pos_int(router, "top", rt), scale=_number(router, "scale", rt),
                                  groups=_pos_int(g, "count", rt + "groups.") if g is not None else 1,
                                  keep=_pos_int(g, "keep", rt + "groups.") if g is not None else 1)
            if c.experts % c.groups:
                raise ConfigError(f"{rt}groups.count={c.groups} must divide the {c.experts} experts")
            if c.keep > c.groups:
                raise ConfigError(f"{rt}groups.keep={c.keep} exceeds groups.count={c.groups}")
            if c.top > c.experts // c.groups * c.keep:
                raise ConfigError(f"{rt}top={c.top} exceeds the {c.experts // c.groups * c.keep} experts of the groups kept")
            return c
        raise ConfigError(f"{at}kind={kind!r} is not a feed-forward of this design (dense, moe)")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> Dict[str, Any]:
        layers = []
        for m, f in zip(self.mixers, self.mlps):
            mixer = {k: v.to_dict() if isinstance(v, RotaryConfig) else v for k, v in vars(m).items()}
            mlp: Optional[Dict[str, Any]] = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top, "scale": f.scale,
                                                                         "groups": {"count": f.groups, "keep": f.keep}}}
            layers.append({"type": m.KIND, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                             "max_positions": self.max_positions, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                             "logit_scale": self.logit_scale, "layers": layers}
        if self.loop is not None:
            d["loop"] = dict(vars(self.loop))
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
        return tuple(LayerRun(i) for i in [*range(a), *(list(range(a, b)) * self.loop.times), *range(b, n)])

    def model_spec(self) -> ModelSpec:
        D, eps, S = self.hidden_size, self.norm_eps, self.streams
        norm = PartSpec("stream_rmsnorm", {"size": D, "streams": S, "eps": eps, "leaf": ""})
        block = PartSpec("stream_residual", {"hidden_size": D, "streams": S, "multiplier": self.residual_mult, "mixer_name": "mix",
                                             "feed_forward_name": "mlp", "norm_names": ("norm1", "norm2"), "connection_names": ("hc1", "hc2"),
                                             "gate_names": ("rg1", "rg2")})
        layers = []
        for i, (m, f) in enumerate(zip(self.mixers, self.mlps)):
            if isinstance(m, DifferenceAttentionConfig):
                mixer = PartSpec("difference_attention", {
                    "hidden_size": D, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "qk_dim": m.dim, "v_dim": m.vdim, "scale": m.scale,
                    "diff": m.diff, "norm_eps": eps, "position_encoding": m.rot.part(interleaved=True)})
            elif isinstance(m, MemoryConfig):
                mixer = PartSpec("forget_memory", {"hidden_size": D, "num_heads": m.heads, "qk_dim": m.dim, "v_dim": m.vdim, "norm_eps": eps})
            else:
                mixer = PartSpec("latent_attention", {
                    "hidden_size": D, "num_heads": m.heads, "nope_dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim, "kv_rank": m.kv_rank,
                    "scale": m.scale, "norm_eps": eps, "output_gate": True, "position_encoding": m.rot.part(interleaved=False)})
            parts = {"mixer": mixer, "mixer_norm": norm}
            if f is not None:
                parts["feed_forward_norm"] = norm
                if f.kind == "dense":
                    parts["feed_forward"] = PartSpec("gated_dense", {"hidden_size": D, "intermediate_size": f.ff, "activation": "silu", "biases": True})
                else:
                    parts["feed_forward"] = PartSpec("routed_experts", {
                        "hidden_size": D, "num_experts": f.experts, "top_k": f.top, "expert_size": f.ff, "route_scale": f.scale,
                        "routing": "sigmoid", "activation": "gelu", "groups": (f.groups, f.keep)})
            layers.append(LayerSpec(prefix=f"l{i}", block=block, parts=parts))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=D, vocab_size=self.vocab_size, max_positions=self.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab_size, "hidden_size": D, "leaf": "", "streams": S,
                                                   "position_table": "pos", "max_positions": self.max_positions}),
            layers=tuple(layers), order=self.order(), final_norm=norm.with_params(scale=self.logit_scale),
            lm_head=PartSpec("lm_head", {"vocab_size": self.vocab_size, "hidden_size": D, "leaf": "", "tied_to": "embed"}),
            embedding_prefix="embed", final_norm_prefix="final.norm", lm_head_prefix="head")
        spec.validate()
        return spec

    @staticmethod
    def canonical_tensor_name(name: str) -> str:
        return name

    def ignorable_tensor(self, name: str) -> bool:
        """What is stored for the feed-forward sublayer of a layer that does not have one."""
        layer, _, rest = name.partition(".")
        return rest.split(".")[0] in ("norm2", "hc2", "rg2") and any(f is None and layer == f"l{i}" for i, f in enumerate(self.mlps))
