"""Tiny Vaderax configurations and weights for the tests.

The configurations differ from one another in every size, in the order of the layers and in what a layer has: models that
start with either mixer, a model without any attention (no pages at all), layers without a feed-forward, dense and routed
feed-forwards, routers with and without identity experts, with one group, with groups of which one, some or all are kept, all
experts chosen, grouped query/key heads and one per head, query/key and value sizes that differ, fewer rotated coordinates
than a head is wide, one tap and five, loops over the whole model, over one layer, over the first or the last layers, a loop of
one pass and none, sizes that are no multiples of 8 or 16.

Weights are drawn so that activations stay of order one through the layers (matrices with variance 1 / inputs).
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict

import torch

from llmengine_b200.weights import write_safetensors


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, scale, base=10000.0, dims=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
            "rot": {"base": base, "dims": dim if dims is None else dims}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=None, groups=None):
    r = {"experts": experts, "top": top}
    if identity is not None:
        r["identity"] = identity
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, eps, scale, layers, loop=None):
    d = {"architecture": "Vaderax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


# sizes the tensor-core kernels take; starts with a delta layer inside the loop; three groups of which two are kept
TINY_A = model(103, 64, 1e-5, 7.0, [
    layer("delta", delta(4, 2, 16, 32, 4), dense(96)),
    layer("attention", attention(4, 2, 32, 32, 0.2, base=500.0, dims=16), moe(7, 3, 24, identity=2, groups=(3, 2))),
    layer("delta", delta(2, 2, 32, 16, 2), moe(4, 1, 32, identity=4, groups=(4, 3))),
    layer("attention", attention(6, 2, 16, 48, 0.3, base=90.0)),
], loop=(0, 2, 3))

# sizes that are no multiples of 8: the plain kernels everywhere; starts with attention; one tap and five; no identity experts, no
# groups, all experts chosen; the loop is one layer
TINY_B = model(71, 52, 1e-6, 3.0, [
    layer("attention", attention(3, 1, 12, 10, 0.3, base=40.0, dims=6), dense(44)),
    layer("delta", delta(3, 1, 6, 5, 5), moe(3, 3, 20)),
    layer("delta", delta(2, 1, 20, 7, 1)),
    layer("attention", attention(2, 2, 20, 6, 0.2, base=2000.0), moe(5, 2, 12, identity=1, groups=(3, 3))),
], loop=(1, 2, 2))

# no attention at all: the engine then has states and no pages; the loop ends the model
ONLY_DELTA = model(83, 48, 1e-5, 2.0, [
    layer("delta", delta(2, 1, 8, 16, 3), dense(64)),
    layer("delta", delta(3, 3, 40, 9, 2)),
], loop=(1, 2, 3))

# attention alone, the whole model in a loop, all of them a page group of their own
ONLY_ATTENTION = model(61, 40, 1e-5, 5.0, [
    layer("attention", attention(4, 1, 16, 16, 0.35, base=100.0, dims=8), moe(4, 2, 16, identity=2, groups=(2, 1))),
], loop=(0, 1, 2))

# a loop of a single pass is no loop
ONE_PASS = model(47, 24, 1e-5, 4.0, [
    layer("delta", delta(2, 2, 8, 8, 4), moe(2, 2, 12, identity=2, groups=(2, 2))),
    layer("attention", attention(2, 1, 8, 8, 0.4, base=30.0, dims=4), dense(20)),
], loop=(0, 2, 1))


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Every tensor of a model of this configuration, by the design's naming."""
    D, V = cfg["width"], cfg["vocab"]
    s: Dict[str, tuple] = {"embed": (V, D), "final.norm": (D,), "final.norm.b": (D,), "head": (V, D)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = s[p + "norm1.b"] = (D,)
        H, G = m["heads"], m["kv_heads"]
        s.update({p + "mix.q": ((G if L["type"] == "delta" else H) * m["dim"], D), p + "mix.k": (G * m["dim"], D),
                  p + "mix.v": ((H if L["type"] == "delta" else G) * m["vdim"], D), p + "mix.g": (H * m["vdim"], D),
                  p + "mix.o": (D, H * m["vdim"])})
        if L["type"] == "delta":
            s.update({p + "mix.q.conv": (G * m["dim"], m["conv"]), p + "mix.k.conv": (G * m["dim"], m["conv"]),
                      p + "mix.v.conv": (H * m["vdim"], m["conv"]), p + "mix.b": (H, D), p + "mix.a": (H, D), p + "mix.A_log": (H,),
                      p + "mix.dt_bias": (H,), p + "mix.norm": (m["vdim"],)})
        mlp = L["mlp"]
        if mlp is None:
            continue
        s[p + "norm2"] = s[p + "norm2.b"] = (D,)
        if mlp["kind"] == "dense":
            s.update({p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
        else:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            n = E + mlp["router"].get("identity", 0)
            s.update({p + "mlp.router": (n, D), p + "mlp.correction": (n,)})
            for e in range(E):
                s.update({p + f"mlp.e{e}.up": (ff, D), p + f"mlp.e{e}.down": (D, ff)})
    return s


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)              # gains (the model's, and those behind the delta rule)
        elif leaf == "b" and len(shape) == 1:
            t = 0.3 * torch.randn(shape, generator=g)                     # biases of the norms
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif leaf == "A_log":
            t = -1.0 + torch.randn(shape, generator=g)
        elif leaf == "dt_bias":
            t = -2.0 + torch.randn(shape, generator=g)                    # decays that mostly keep
        elif leaf == "correction":
            t = 0.2 * torch.randn(shape, generator=g)                     # moves choices, and makes choice scores negative
        elif leaf == "down":
            t = torch.randn(shape, generator=g) / math.sqrt(1.5 * shape[-1])      # relu(z)^2 of z ~ N(0, 1) has a mean square of 1.5
        elif name == "embed":
            t = torch.randn(shape, generator=g) / cfg["embedding"]["scale"]
        elif leaf == "router":
            t = 1.5 * torch.randn(shape, generator=g) / math.sqrt(shape[-1])      # routers that decide
        else:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def make_vaderax_dir(path: str, cfg: dict, seed: int, change=None) -> str:
    """A model folder with random weights; `change(weights)` may edit them (tests that make one key stand out)."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    w = make_weights(cfg, seed)
    if change is not None:
        change(w)
    write_safetensors(os.path.join(path, "model.safetensors"), w)
    return path
