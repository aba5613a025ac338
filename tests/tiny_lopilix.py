"""Tiny Lopilix configurations and weights for the tests.

The configurations differ from one another in every size, in the order of the layers and in what a layer has: models that
start with each of the mixers, a model without any attention (no pages at all), one of each attention alone, layers without a
feed-forward, dense and routed feed-forwards, routers without groups, with groups of which one, some or all are kept, groups of
one expert, all experts chosen, one stream and five, heads that share keys and values and heads that do not, value sizes that
are and are not twice the query size, fewer rotated coordinates than a head is wide, stretched frequencies and plain ones,
latent sizes the tensor-core kernel takes and others, loops over the whole model, over one layer, over the last layers, a loop of
one pass and none, sizes that are no multiples of 4, 8 or 16.

Weights are drawn so that activations stay of order one through the layers (matrices with variance 1 / inputs).
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict

import torch

from llmengine_b200.weights import write_safetensors


def attention(heads, kv_heads, dim, vdim, scale, diff, base=10000.0, dims=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff,
            "rot": {"base": base, "dims": dim if dims is None else dims}}


def memory(heads, dim, vdim):
    return {"heads": heads, "dim": dim, "vdim": vdim}


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, scaling=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": rot}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=1.0, groups=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, streams, positions, eps, mult, logit_scale, layers, loop=None):
    d = {"architecture": "Lopilix", "vocab": vocab, "width": width, "streams": streams, "max_positions": positions, "norm": {"eps": eps},
         "residual_mult": mult, "logit_scale": logit_scale, "layers": layers}
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


# sizes the tensor-core kernels take; starts with the memory inside the loop; three groups of which two are kept
TINY_A = model(101, 64, 3, 600, 1e-5, 0.8, 1.7, [
    layer("hgrn2", memory(3, 24, 40), moe(9, 2, 40, 1.5, groups=(3, 2))),
    layer("attention", attention(4, 2, 32, 64, 0.2, 0.35, base=500.0, dims=16), dense(96)),
    layer("latent_attention", latent(3, 16, 8, 24, 64, 0.25, base=300.0, scaling=(8.0, 64, 8.0, 1.0)), moe(8, 3, 32, 0.7, groups=(2, 1))),
    layer("hgrn2", memory(2, 16, 16), dense(48)),
], loop=(0, 2, 2))

# sizes that are no multiples of 4: the plain kernels everywhere; one stream; starts with the latent; the loop is one layer
TINY_B = model(73, 50, 1, 300, 1e-6, 1.3, 0.4, [
    layer("latent_attention", latent(2, 10, 6, 7, 30, 0.3, base=50.0), dense(44)),
    layer("attention", attention(3, 1, 10, 6, 0.3, 0.7, base=40.0, dims=6), moe(5, 2, 18, 2.5)),
    layer("hgrn2", memory(3, 5, 7)),
    layer("attention", attention(2, 2, 14, 22, 0.25, 0.2, base=900.0), moe(6, 6, 14, 1.0, groups=(3, 3))),
], loop=(1, 2, 3))

# no attention at all: the engine then has states and no pages; five streams; the loop ends the model
ONLY_MEMORY = model(83, 40, 5, 200, 1e-5, 0.6, 2.0, [
    layer("hgrn2", memory(2, 8, 16), dense(64)),
    layer("hgrn2", memory(1, 70, 12), moe(4, 1, 24, 1.2, groups=(4, 2))),
], loop=(1, 2, 2))

# each attention alone, the whole model in a loop
ONLY_ATTENTION = model(61, 48, 2, 500, 1e-5, 0.9, 1.0, [
    layer("attention", attention(6, 3, 16, 32, 0.35, 0.5, base=100.0, dims=8), moe(4, 2, 16, 2.0)),
], loop=(0, 1, 3))

ONLY_LATENT = model(67, 32, 4, 500, 1e-5, 1.0, 3.0, [
    layer("latent_attention", latent(4, 8, 16, 16, 128, 0.3, base=1000.0, scaling=(2.0, 128, 16.0, 2.0))),
    layer("latent_attention", latent(2, 24, 4, 8, 40, 0.4, base=20.0), dense(40)),
])

# a loop of a single pass is no loop
ONE_PASS = model(47, 24, 2, 128, 1e-5, 0.5, 0.8, [
    layer("hgrn2", memory(2, 12, 8), moe(6, 2, 12, 1.0, groups=(2, 2))),
    layer("attention", attention(2, 1, 8, 16, 0.4, 0.6, base=30.0, dims=4), dense(20)),
], loop=(0, 2, 1))


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Every tensor of a model of this configuration, by the design's naming."""
    D, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    s: Dict[str, tuple] = {"embed": (V, D), "pos": (cfg["max_positions"], D), "final.norm": (D,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        H = m["heads"]
        for q in ("1",) + (("2",) if L["mlp"] is not None else ()):
            s.update({p + "norm" + q: (D,), p + f"hc{q}.in": (S,), p + f"hc{q}.out": (S,), p + f"hc{q}.mix": (S, S), p + "rg" + q: (D, D),
                      p + f"rg{q}.b": (D,)})
        s[p + "mix.o"] = (D, H * m["vdim"])
        if L["type"] == "attention":
            G, d = m["kv_heads"], m["dim"]
            s.update({p + "mix.q": (2 * H * d, D), p + "mix.k": (2 * G * d, D), p + "mix.v": (G * m["vdim"], D), p + "mix.q.norm": (d,),
                      p + "mix.k.norm": (d,), **{p + "mix." + n: (d,) for n in ("lq1", "lk1", "lq2", "lk2")}})
        elif L["type"] == "hgrn2":
            n = H * m["dim"]
            s.update({p + "mix.q": (n, D), p + "mix.f": (n, D), p + "mix.f.b": (n,), p + "mix.lower": (n,), p + "mix.v": (H * m["vdim"], D),
                      p + "mix.norm": (m["vdim"],)})
        else:
            R = m["kv_rank"]
            s.update({p + "mix.q": (H * (m["dim"] + m["rot_dim"]), D), p + "mix.dkv": (R + m["rot_dim"], D), p + "mix.dkv.norm": (R,),
                      p + "mix.uk": (H * m["dim"], R), p + "mix.uv": (H * m["vdim"], R), p + "mix.g": (H * m["vdim"], D)})
        mlp = L["mlp"]
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ff = mlp["ff"]
            s.update({p + "mlp.gate": (ff, D), p + "mlp.gate.b": (ff,), p + "mlp.up": (ff, D), p + "mlp.up.b": (ff,), p + "mlp.down": (D, ff),
                      p + "mlp.down.b": (D,)})
        else:
            E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
            s[p + "mlp.router"] = (E, D)
            for e in range(E):
                s.update({p + f"mlp.e{e}.up": (ff, D), p + f"mlp.e{e}.down": (D, ff)})
    return s


def make_weights(cfg: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    S = cfg["streams"]
    rnd = lambda shape: torch.randn(shape, generator=g)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.3 * rnd(shape)
        elif leaf == "in":
            t = 1.0 / S + 0.4 * rnd(shape)
        elif leaf == "out":
            t = 1.0 + 0.4 * rnd(shape)
        elif leaf == "mix":
            t = torch.eye(S) * 0.8 + 0.25 * rnd(shape) / math.sqrt(S)                   # streams that stay apart and do talk
        elif leaf == "b":
            t = 0.5 * rnd(shape) + (1.0 if name.endswith("f.b") else 0.0)
        elif leaf == "lower":
            t = 0.9 * torch.rand(shape, generator=g)                                     # gates between the bound and one
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.4 * rnd(shape) / math.sqrt(shape[0]) ** 0.5
        elif leaf == "router":
            t = 1.5 * rnd(shape) / math.sqrt(shape[-1])                                  # routers that decide
        elif name in ("embed", "pos"):
            t = rnd(shape)
        else:
            t = rnd(shape) / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def make_lopilix_dir(path: str, cfg: dict, seed: int, change=None) -> str:
    """A model folder with random weights; `change(weights)` may edit them (tests that make one key stand out)."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    w = make_weights(cfg, seed)
    if change is not None:
        change(w)
    write_safetensors(os.path.join(path, "model.safetensors"), w)
    return path
