"""How a layer arranges its mixer, feed-forward and norms."""
from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch

from ..config.spec import LayerSpec
from ..engine.plan import Plan, StreamUpdate
from .base import (Part, Runtime, WeightSpec, build_part, emit_feed_forward, emit_mixer, emit_norm, register_part,
                   run_alone)


@register_part("block", "prenorm_residual")
class PreNormResidualBlock(Part):
    """x = x + mixer(norm1(x));  x = x + feed_forward(norm2(x))
    (src/model/transformer_graph_builder.cpp:207-274: the un-normed x is the residual).

    The residual stream `x` stays 32-bit.  A contribution is not added where it is produced:
    it travels as `delta` to the next norm, whose kernel adds it to `x` and normalises in one
    pass.  The block reads the parts "mixer", "mixer_norm" and, where the layer has a feed-forward, "feed_forward" and
    "feed_forward_norm" of its layer; the names under which their tensors are stored come with the spec.
    """

    def __init__(self, rt: Runtime, prefix: str, layer: LayerSpec, mixer_name: str = "mixer",
                 feed_forward_name: str = "feed_forward", mixer_norm_name: str = "mixer_norm",
                 feed_forward_norm_name: str = "feed_forward_norm"):
        super().__init__(rt, prefix)
        missing = [n for n in ("mixer", "mixer_norm") if n not in layer.parts]
        has_ffn = "feed_forward" in layer.parts
        if has_ffn and "feed_forward_norm" not in layer.parts:
            missing.append("feed_forward_norm")
        if missing:
            raise ValueError(f"layer {prefix!r}: a prenorm_residual block needs the parts {', '.join(missing)}")
        self.mixer_norm = build_part("norm", layer.parts["mixer_norm"], rt, self.name(mixer_norm_name))
        self.mixer = build_part("mixer", layer.parts["mixer"], rt, self.name(mixer_name))
        self.ffn_norm = self.ffn = None
        if has_ffn:
            self.ffn_norm = build_part("norm", layer.parts["feed_forward_norm"], rt, self.name(feed_forward_norm_name))
            self.ffn = build_part("feed_forward", layer.parts["feed_forward"], rt, self.name(feed_forward_name))
        self.parts = tuple(p for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if p is not None)
        self.capture_safe = all(p.capture_safe and hasattr(p, "emit") for p in self.parts)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for p in self.parts:
            out.update(p.weight_specs())
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            p.load_weights({n: tensors[n] for n in p.weight_specs()})

    def cache_spec(self):
        return self.mixer.cache_spec()

    def emit(self, plan: Plan, x: torch.Tensor, delta: Optional[torch.Tensor], cache) -> Tuple[torch.Tensor, torch.Tensor]:
        hidden = x.shape[1]
        h = emit_norm(plan, self.mixer_norm, x, delta=delta)
        a = emit_mixer(plan, self.mixer, h, cache, hidden)
        if self.ffn is None:
            return x, a
        h = emit_norm(plan, self.ffn_norm, x, delta=a)
        return x, emit_feed_forward(plan, self.ffn, h, hidden)

    def forward(self, x: torch.Tensor, delta: Optional[torch.Tensor], batch, cache) -> Tuple[torch.Tensor, torch.Tensor]:
        plan = Plan()
        x, out = self.emit(plan, x, delta, cache)
        run_alone(self.rt, plan, batch)
        return x, out[: x.shape[0]]


@register_part("block", "parallel_residual")
class ParallelResidualBlock(Part):
    """h = norm(x);  x = x + (mixer(h) + feed_forward(h)): one norm, both sublayers read its output.  A layer may
    have no feed-forward.  With a "token_side" part, that part follows on the updated x (and does the addition of
    the sublayers' contributions itself, in the same pass).

    Options of other designs: with a part "feed_forward_norm" the feed-forward reads a norm of its own of the same x
    (x = x + mixer(norm(x)) + feed_forward(feed_forward_norm(x))); with `mixer_scale_name` / `feed_forward_scale_name`
    each sublayer's result is multiplied, column by column, by a learned vector of the stream's width (tensors of those
    names below the layer's prefix) before the sum.

    The block reads the parts "norm", "mixer" and, where the layer has them, "feed_forward", "feed_forward_norm" and
    "token_side".
    """

    def __init__(self, rt: Runtime, prefix: str, layer: LayerSpec, norm_name: str = "norm", mixer_name: str = "mixer",
                 feed_forward_name: str = "feed_forward", token_side_name: str = "token_side",
                 feed_forward_norm_name: str = "feed_forward_norm", mixer_scale_name: Optional[str] = None,
                 feed_forward_scale_name: Optional[str] = None, hidden_size: Optional[int] = None):
        super().__init__(rt, prefix)
        missing = [n for n in ("norm", "mixer") if n not in layer.parts]
        if missing:
            raise ValueError(f"layer {prefix!r}: a parallel_residual block needs the parts {', '.join(missing)}")
        self.norm = build_part("norm", layer.parts["norm"], rt, self.name(norm_name))
        self.mixer = build_part("mixer", layer.parts["mixer"], rt, self.name(mixer_name))
        self.ffn = (build_part("feed_forward", layer.parts["feed_forward"], rt, self.name(feed_forward_name))
                    if "feed_forward" in layer.parts else None)
        self.ffn_norm = (build_part("norm", layer.parts["feed_forward_norm"], rt, self.name(feed_forward_norm_name))
                         if self.ffn is not None and "feed_forward_norm" in layer.parts else None)
        self.side = (build_part("token_side", layer.parts["token_side"], rt, self.name(token_side_name))
                     if "token_side" in layer.parts else None)
        self.scale_names = (mixer_scale_name, feed_forward_scale_name if self.ffn is not None else None)
        if any(self.scale_names) and (hidden_size is None or self.side is not None):
            raise ValueError(f"layer {prefix!r}: scale vectors need the stream's width and a block without a token side input")
        self.hidden = None if hidden_size is None else int(hidden_size)
        self.scales = [None, None]
        self.parts = tuple(p for p in (self.norm, self.mixer, self.ffn_norm, self.ffn, self.side) if p is not None)
        self.capture_safe = all(p.capture_safe and hasattr(p, "emit") for p in self.parts)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for p in self.parts:
            out.update(p.weight_specs())
        for n in self.scale_names:
            if n:
                out[self.name(n)] = WeightSpec((self.hidden,), role="vector", init="gain")
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            p.load_weights({n: tensors[n] for n in p.weight_specs()})
        self.scales = [tensors[self.name(n)].float().contiguous() if n else None for n in self.scale_names]

    def tied_tensors(self) -> Dict[str, str]:
        out: Dict[str, str] = {}
        for p in self.parts:
            out.update(p.tied_tensors())
        return out

    def receive_tied(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            own = p.tied_tensors()
            if own:
                p.receive_tied({n: tensors[n] for n in own})

    def cache_spec(self):
        return self.mixer.cache_spec()

    def emit(self, plan: Plan, x: torch.Tensor, delta: Optional[torch.Tensor], cache):
        hidden = x.shape[1]
        h2 = None
        if self.ffn_norm is not None and hasattr(self.norm, "pairs_with") and self.norm.pairs_with(self.ffn_norm):
            h, h2 = self.norm.emit_pair(plan, self.ffn_norm, x, delta=delta)      # both norms of the same x in one pass
        else:
            h = emit_norm(plan, self.norm, x, delta=delta)
        a = emit_mixer(plan, self.mixer, h, cache, hidden)
        b = None
        if self.ffn is not None:
            # a second norm of the same x goes to a workspace of its own: the mixer's input may still be needed
            if h2 is not None:
                pass
            elif self.ffn_norm is None:
                h2 = h
            elif hasattr(self.ffn_norm, "emit"):
                h2 = self.ffn_norm.emit(plan, x, out_name="normed_second")
            else:
                h2 = emit_norm(plan, self.ffn_norm, x)
            b = emit_feed_forward(plan, self.ffn, h2, hidden)
        if self.side is not None:
            self.side.emit(plan, x, a, b)
            return x, None
        if b is None and self.scales[0] is None:
            return x, a                       # the next norm adds it
        plan.residual_add(x, a, b, a_scale=self.scales[0], b_scale=self.scales[1] if b is not None else None)
        return x, None

    def forward(self, x: torch.Tensor, delta: Optional[torch.Tensor], batch, cache):
        plan = Plan()
        x, out = self.emit(plan, x, delta, cache)
        run_alone(self.rt, plan, batch)
        return x, None if out is None else out[: x.shape[0]]


@register_part("block", "postnorm_residual")
class PostNormResidualBlock(Part):
    """x = x + norm1(mixer(x));  x = x + norm2(feed_forward(x)): the norms stand on the sublayers' OUTPUTS, and the
    sublayers read the residual stream itself.  A layer may have no feed-forward (and then no second norm).

    The stream is 32-bit.  Where the matrix products take another type, the kernel that adds a normed contribution
    also writes the new stream in that type, which is what the next sublayer reads.  The block reads the parts
    "mixer", "mixer_norm" and, where the layer has them, "feed_forward" and "feed_forward_norm" (norm parts with a
    gain vector and an eps)."""

    def __init__(self, rt: Runtime, prefix: str, layer: LayerSpec, mixer_name: str = "mixer",
                 feed_forward_name: str = "feed_forward", mixer_norm_name: str = "mixer_norm",
                 feed_forward_norm_name: str = "feed_forward_norm"):
        super().__init__(rt, prefix)
        missing = [n for n in ("mixer", "mixer_norm") if n not in layer.parts]
        if "feed_forward" in layer.parts and "feed_forward_norm" not in layer.parts:
            missing.append("feed_forward_norm")
        if missing:
            raise ValueError(f"layer {prefix!r}: a postnorm_residual block needs the parts {', '.join(missing)}")
        self.mixer = build_part("mixer", layer.parts["mixer"], rt, self.name(mixer_name))
        self.mixer_norm = build_part("norm", layer.parts["mixer_norm"], rt, self.name(mixer_norm_name))
        has_ffn = "feed_forward" in layer.parts
        self.ffn = build_part("feed_forward", layer.parts["feed_forward"], rt, self.name(feed_forward_name)) if has_ffn else None
        self.ffn_norm = build_part("norm", layer.parts["feed_forward_norm"], rt, self.name(feed_forward_norm_name)) if has_ffn else None
        self.parts = tuple(p for p in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if p is not None)
        for n in (self.mixer_norm, self.ffn_norm):
            if n is not None and not (hasattr(n, "gain") and hasattr(n, "eps")):
                raise ValueError(f"layer {prefix!r}: the norm on a sublayer's output needs a gain vector and an eps")
        self.capture_safe = all(p.capture_safe and hasattr(p, "emit") for p in (self.mixer, self.ffn) if p is not None)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for p in self.parts:
            out.update(p.weight_specs())
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            p.load_weights({n: tensors[n] for n in p.weight_specs()})

    def cache_spec(self):
        return self.mixer.cache_spec()

    def _input(self, plan: Plan, x: torch.Tensor) -> torch.Tensor:
        """The stream as a sublayer reads it: itself in the 32-bit engine, else its copy in the product type."""
        rt = self.rt
        if rt.dtype == torch.float32:
            return x
        h = plan.copy_of(x)
        if h is None:
            h = rt.workspace("stream_copy", x.shape[1], rt.dtype)
            plan.postnorm(x, None, None, 0.0, copy=h)
        return h

    def emit(self, plan: Plan, x: torch.Tensor, delta: Optional[torch.Tensor], cache):
        rt = self.rt
        hidden = x.shape[1]
        if delta is not None:
            plan.residual_add(x, delta)
        copy = None if rt.dtype == torch.float32 else rt.workspace("stream_copy", hidden, rt.dtype)
        a = emit_mixer(plan, self.mixer, self._input(plan, x), cache, hidden)
        plan.postnorm(x, a, self.mixer_norm.gain, self.mixer_norm.eps, copy=copy)
        if self.ffn is not None:
            b = emit_feed_forward(plan, self.ffn, self._input(plan, x), hidden)
            plan.postnorm(x, b, self.ffn_norm.gain, self.ffn_norm.eps, copy=copy)
        return x, None

    def forward(self, x: torch.Tensor, delta: Optional[torch.Tensor], batch, cache):
        plan = Plan()
        x, _ = self.emit(plan, x, delta, cache)
        run_alone(self.rt, plan, batch)
        return x, None


@register_part("block", "sandwich_residual")
class SandwichResidualBlock(Part):
    """x = x + norm1b(mixer(norm1(x)));  x = x + norm2b(feed_forward(norm2(x))): a norm before AND after each sublayer.
    A layer may have no feed-forward (and then neither of its norms).

    The stream is 32-bit.  The norm before a sublayer writes its input in the type of the products; the norm behind it
    is the kernel that norms a sublayer's output and adds it to the stream in one pass.  The block reads the parts
    "mixer", "mixer_norm", "mixer_out_norm" and, where the layer has a feed-forward, "feed_forward", "feed_forward_norm"
    and "feed_forward_out_norm"."""

    def __init__(self, rt: Runtime, prefix: str, layer: LayerSpec, mixer_name: str = "mixer", feed_forward_name: str = "feed_forward",
                 mixer_norm_name: str = "mixer_norm", mixer_out_norm_name: str = "mixer_out_norm",
                 feed_forward_norm_name: str = "feed_forward_norm", feed_forward_out_norm_name: str = "feed_forward_out_norm"):
        super().__init__(rt, prefix)
        has_ffn = "feed_forward" in layer.parts
        need = ["mixer", "mixer_norm", "mixer_out_norm"] + (["feed_forward_norm", "feed_forward_out_norm"] if has_ffn else [])
        missing = [n for n in need if n not in layer.parts]
        if missing:
            raise ValueError(f"layer {prefix!r}: a sandwich_residual block needs the parts {', '.join(missing)}")
        self.mixer_norm = build_part("norm", layer.parts["mixer_norm"], rt, self.name(mixer_norm_name))
        self.mixer = build_part("mixer", layer.parts["mixer"], rt, self.name(mixer_name))
        self.mixer_out_norm = build_part("norm", layer.parts["mixer_out_norm"], rt, self.name(mixer_out_norm_name))
        self.ffn = self.ffn_norm = self.ffn_out_norm = None
        if has_ffn:
            self.ffn_norm = build_part("norm", layer.parts["feed_forward_norm"], rt, self.name(feed_forward_norm_name))
            self.ffn = build_part("feed_forward", layer.parts["feed_forward"], rt, self.name(feed_forward_name))
            self.ffn_out_norm = build_part("norm", layer.parts["feed_forward_out_norm"], rt, self.name(feed_forward_out_norm_name))
        self.parts = tuple(p for p in (self.mixer_norm, self.mixer, self.mixer_out_norm, self.ffn_norm, self.ffn, self.ffn_out_norm)
                           if p is not None)
        for n in (self.mixer_out_norm, self.ffn_out_norm):
            if n is not None and not (hasattr(n, "gain") and hasattr(n, "eps")):
                raise ValueError(f"layer {prefix!r}: the norm on a sublayer's output needs a gain vector and an eps")
        self.capture_safe = all(p.capture_safe and hasattr(p, "emit") for p in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn)
                                if p is not None)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for p in self.parts:
            out.update(p.weight_specs())
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            p.load_weights({n: tensors[n] for n in p.weight_specs()})

    def cache_spec(self):
        return self.mixer.cache_spec()

    def emit(self, plan: Plan, x: torch.Tensor, delta: Optional[torch.Tensor], cache):
        hidden = x.shape[1]
        h = emit_norm(plan, self.mixer_norm, x, delta=delta)
        a = emit_mixer(plan, self.mixer, h, cache, hidden)
        plan.postnorm(x, a, self.mixer_out_norm.gain, self.mixer_out_norm.eps)
        if self.ffn is not None:
            h = emit_norm(plan, self.ffn_norm, x)
            b = emit_feed_forward(plan, self.ffn, h, hidden)
            plan.postnorm(x, b, self.ffn_out_norm.gain, self.ffn_out_norm.eps)
        return x, None

    def forward(self, x: torch.Tensor, delta: Optional[torch.Tensor], batch, cache):
        plan = Plan()
        x, _ = self.emit(plan, x, delta, cache)
        run_alone(self.rt, plan, batch)
        return x, None


@register_part("block", "stream_residual")
class StreamResidualBlock(Part):
    """Hyper-connections: the residual stream is S streams x_1 .. x_S side by side ([T, S D], 32-bit).  Each sublayer q (the mixer,
    then the feed-forward, where the layer has one) reads h = norm_q(sum_s in_q[s] x_s); its result, gated, goes into all of them:
        y = sublayer(h) * sigmoid(W_q h + b_q);   x_t <- sum_s mix_q[s, t] x_s + multiplier * out_q[t] * y  (all from the old ones).

    Tensors below the layer's prefix: <connection>.in [S], .out [S], .mix [S, S] ([from, to]); the gate's <gate> [D, D] and
    <gate>.b [D]; the norms' under their names.  A sublayer's result is not written where it is produced: it travels as a
    `StreamUpdate` to the next norm, whose kernel updates the streams, sums what its own sublayer reads and norms it in one
    pass.  The block reads the parts "mixer", "mixer_norm" and, where the layer has them, "feed_forward" and
    "feed_forward_norm", the norms of a kind that takes a stream's read weights (`stream_rmsnorm`)."""

    def __init__(self, rt: Runtime, prefix: str, layer: LayerSpec, hidden_size: int, streams: int, multiplier: float = 1.0,
                 mixer_name: str = "mixer", feed_forward_name: str = "feed_forward",
                 norm_names: Tuple[str, str] = ("mixer_norm", "feed_forward_norm"),
                 connection_names: Tuple[str, str] = ("mixer_connection", "feed_forward_connection"),
                 gate_names: Tuple[str, str] = ("mixer_gate", "feed_forward_gate")):
        super().__init__(rt, prefix)
        missing = [n for n in ("mixer", "mixer_norm") if n not in layer.parts]
        has_ffn = "feed_forward" in layer.parts
        if has_ffn and "feed_forward_norm" not in layer.parts:
            missing.append("feed_forward_norm")
        if missing:
            raise ValueError(f"layer {prefix!r}: a stream_residual block needs the parts {', '.join(missing)}")
        self.hidden, self.streams, self.multiplier = int(hidden_size), int(streams), float(multiplier)
        self.norms = [build_part("norm", layer.parts["mixer_norm"], rt, self.name(norm_names[0]))]
        self.mixer = build_part("mixer", layer.parts["mixer"], rt, self.name(mixer_name))
        self.ffn = None
        if has_ffn:
            self.norms.append(build_part("norm", layer.parts["feed_forward_norm"], rt, self.name(norm_names[1])))
            self.ffn = build_part("feed_forward", layer.parts["feed_forward"], rt, self.name(feed_forward_name))
        self.parts = tuple(p for p in (*self.norms, self.mixer, self.ffn) if p is not None)
        self.sublayers = tuple(p for p in (self.mixer, self.ffn) if p is not None)
        n = len(self.norms)
        self.connections, self.gates = tuple(connection_names[:n]), tuple(gate_names[:n])
        self.capture_safe = all(p.capture_safe and hasattr(p, "emit") for p in self.parts)
        self.read, self.mix, self.put, self.w_gate, self.b_gate = [], [], [], [], []

    def weight_specs(self) -> Dict[str, WeightSpec]:
        out: Dict[str, WeightSpec] = {}
        for p in self.parts:
            out.update(p.weight_specs())
        S, D = self.streams, self.hidden
        for c, g in zip(self.connections, self.gates):
            out[self.name(c + ".in")] = WeightSpec((S,), role="vector", init="gain")
            out[self.name(c + ".out")] = WeightSpec((S,), role="vector", init="gain")
            out[self.name(c + ".mix")] = WeightSpec((S, S), role="vector")
            out[self.name(g)] = WeightSpec((D, D))
            out[self.name(g + ".b")] = WeightSpec((D,), role="vector")
        return out

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        for p in self.parts:
            p.load_weights({n: tensors[n] for n in p.weight_specs()})
        f = lambda n: tensors[self.name(n)].float().contiguous()
        self.read, self.mix = [f(c + ".in") for c in self.connections], [f(c + ".mix") for c in self.connections]
        self.put = [f(c + ".out") * self.multiplier for c in self.connections]
        self.w_gate, self.b_gate = [tensors[self.name(g)].contiguous() for g in self.gates], [f(g + ".b") for g in self.gates]
        for q, part in enumerate(self.sublayers):
            if part.carries_rows:                     # the gate reads the sublayer's own input: it rides in its first product
                part.carry_rows(self.w_gate[q])
                self.w_gate[q] = None

    def cache_spec(self):
        return self.mixer.cache_spec()

    def _result(self, plan: Plan, q: int, h: torch.Tensor, y: torch.Tensor) -> StreamUpdate:
        """Sublayer q's result `y` on its way into the streams, with what its gate is made from: columns of the sublayer's first
        product, or a product of its own where the sublayer carries no rows."""
        gate = self.sublayers[q].carried
        if self.w_gate[q] is not None:
            gate = self.rt.workspace("sublayer_gate", self.hidden, self.rt.dtype)
            plan.linear(h, self.w_gate[q], gate)
        return StreamUpdate(y=y, gate=gate, bias=self.b_gate[q], mix=self.mix[q], put=self.put[q])

    def emit(self, plan: Plan, x: torch.Tensor, delta: Optional[StreamUpdate], cache):
        h = self.norms[0].emit(plan, x, delta=delta, read=self.read[0])
        delta = self._result(plan, 0, h, emit_mixer(plan, self.mixer, h, cache, self.hidden))
        if self.ffn is not None:
            h = self.norms[1].emit(plan, x, delta=delta, read=self.read[1])
            delta = self._result(plan, 1, h, emit_feed_forward(plan, self.ffn, h, self.hidden))
        return x, delta

    def forward(self, x: torch.Tensor, delta: Optional[StreamUpdate], batch, cache):
        plan = Plan()
        x, delta = self.emit(plan, x, delta, cache)
        plan.stream_norm(x, streams=self.streams, read=None, gain=None, eps=0.0, out=None, update=delta)
        run_alone(self.rt, plan, batch)
        return x, None
