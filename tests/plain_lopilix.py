"""The plain implementation of the Lopilix design: whole sequences, no cache, no chunks, one function per mechanism,
elementary tensor arithmetic on the CPU; the recurrence runs token by token.

It shares no code with the engine: it reads config.json and model.safetensors itself.  `round_to` rounds to bfloat16
where the engine's bfloat16 path stores bfloat16 (the inputs of the matrix products, projections, cached rows); the
arithmetic itself is 32-bit (or 64-bit with `wide`).

Notation: D width, T tokens, S streams, H heads, G key/value heads, d query/key size per head (and map), P value size per
head, R latent size, E experts.
"""
from __future__ import annotations

import json
import math
import os
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from plain_bepuzen import read_safetensors


def _r(x: torch.Tensor, round_to: Optional[torch.dtype]) -> torch.Tensor:
    return x if round_to is None else x.to(round_to).to(x.dtype)


# --------------------------------------------------------------------- small pieces
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    """z times the normal distribution's share below z."""
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> Tuple[List[float], float]:
    """(angle per position of every pair, factor on cosine and sine): base^(-2i/dims); stretched (`scaling`): a pair that makes
    many turns over the original length keeps its frequency, one that makes few gets it divided by the factor, a ramp between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    pair_with_turns = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(pair_with_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_with_turns(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        slow = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / scaling["factor"] * slow + v * (1.0 - slow))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def _angles(positions: torch.Tensor, freq: Sequence[float], amplitude: float, dtype) -> Tuple[torch.Tensor, torch.Tensor]:
    f = torch.tensor(list(freq), dtype=torch.float64).to(torch.float32).to(dtype)
    a = positions.to(dtype)[:, None] * f[None, :]
    return (torch.cos(a) * amplitude)[:, None, :], (torch.sin(a) * amplitude)[:, None, :]


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, d]: among the first rot.dims coordinates, 2i pairs with 2i + 1: (u, v) -> (u cos - v sin, v cos + u sin)."""
    n = rot["dims"]
    c, s = _angles(positions, *frequencies(n, rot["base"], rot.get("scaling")), x.dtype)
    out = x.clone()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = u * c - v * s, v * c + u * s
    return out


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """The same turn with the pairs (i, i + dims / 2)."""
    n, half = rot["dims"], rot["dims"] // 2
    c, s = _angles(positions, *frequencies(n, rot["base"], rot.get("scaling")), x.dtype)
    u, v = x[..., :half], x[..., half:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    """Softmax of s [..., i, j] over j <= i."""
    T = s.shape[-1]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


# --------------------------------------------------------------------- mixers
def difference_weight(w, pre, diff: float) -> torch.Tensor:
    """The layer's lambda: exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    return torch.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - torch.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff


def difference_attention(h, w, pre, m, eps, positions, round_to):
    """Two causal softmaxes per head over the same values, each with queries and keys of its own (normed per head and map with
    a weight, then rotated): o = a1 - lambda a2, divided by its root mean square, times 1 - diff.  Query head a reads key and
    value head a // (H / G).  Returns [T, H P]."""
    H, G, d, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, rep = h.shape[0], m["heads"] // m["kv_heads"]
    proj = lambda n: _r(h @ w[pre + n].t(), round_to)
    finish = lambda n, heads: _r(rotate_neighbours(unit_rms(proj(n).view(T, heads * 2, d), eps) * w[pre + n + ".norm"], positions, m["rot"]),
                                 round_to).view(T, heads, 2, d)
    q, k = finish("q", H), finish("k", G).repeat_interleave(rep, 1)
    v = proj("v").view(T, G, P).repeat_interleave(rep, 1)
    maps = [_r(torch.einsum("aij,jap->iap", causal_softmax(torch.einsum("iad,jad->aij", q[:, :, c], k[:, :, c]) * m["scale"]), v), round_to)
            for c in (0, 1)]
    o = maps[0] - difference_weight(w, pre, m["diff"]) * maps[1]
    return (unit_rms(o, eps) * (1.0 - m["diff"])).reshape(T, H * P)


def gated_memory(q, f, v, S=None, sizes=None):
    """q, f [T, H, d], v [T, H, P]: S <- f S + (1 - f) v^T row by row (row c of S decays by f_c and takes (1 - f_c) v), then
    o = S^T q.  Returns o [T, H, P] and S [H, d, P]; `sizes` (a list) receives the norm of every head's S per token."""
    T, H, d = q.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("adp,ad->ap", S, q[t]))
        if sizes is not None:
            sizes.append(S.flatten(1).norm(dim=-1))
    return torch.stack(out), S


def memory_mixer(h, w, pre, m, eps, calls=None):
    """q = silu(W_q h), v = W_v h, f = lower + (1 - lower) sigmoid(W_f h + b_f) per head and channel; the memory; every head's o
    normed over its P values with a weight shared by the heads.  Returns [T, H P].

    `calls` (a list) receives per token how far the model is from a close call: the norm leaves only the direction of S^T q, and
    where q is nearly orthogonal to what the memory holds (a memory of one token: the SIGN of a sum) rounding decides it.
    2.5 sqrt(d) |S^T q| / (|S| |q|), the least over the heads."""
    H, d, P = m["heads"], m["dim"], m["vdim"]
    T, lower = h.shape[0], w[pre + "lower"]
    q = silu(h @ w[pre + "q"].t()).view(T, H, d)
    f = (lower + (1.0 - lower) * torch.sigmoid(h @ w[pre + "f"].t() + w[pre + "f.b"])).view(T, H, d)
    sizes = None if calls is None else []
    o, _ = gated_memory(q, f, (h @ w[pre + "v"].t()).view(T, H, P), sizes=sizes)
    if calls is not None:
        hold = torch.stack(sizes) * q.norm(dim=-1)
        calls.append((2.5 * math.sqrt(d) * (o.norm(dim=-1) / hold.clamp_min(1e-30)).amin(-1)).to(torch.float32))
    return (unit_rms(o, eps) * w[pre + "norm"]).reshape(T, H * P)


def latent_attention(h, w, pre, m, eps, positions, round_to):
    """Keys and values of all heads come from one normed latent per token; beside the unrotated part of a key stands one
    rotated part shared by the heads; the heads, side by side, times sigmoid(W_g h).  Returns [T, H P]."""
    H, d, dr, P, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    q = _r(h @ w[pre + "q"].t(), round_to).view(T, H, d + dr)
    low = _r(h @ w[pre + "dkv"].t(), round_to)
    c = _r(unit_rms(low[:, :R], eps) * w[pre + "dkv.norm"], round_to)
    shared = _r(rotate_halves(low[:, None, R:], positions, m["rot"]), round_to)[:, 0]
    turned = _r(rotate_halves(q[..., d:], positions, m["rot"]), round_to)
    k = (c @ w[pre + "uk"].t()).view(T, H, d)
    v = (c @ w[pre + "uv"].t()).view(T, H, P)
    s = (torch.einsum("iad,jad->aij", q[..., :d], k) + torch.einsum("iad,jd->aij", turned, shared)) * m["scale"]
    o = _r(torch.einsum("aij,jap->iap", causal_softmax(s), v), round_to).reshape(T, H * P)
    return o * torch.sigmoid(_r(h @ w[pre + "g"].t(), round_to))


# --------------------------------------------------------------------- feed-forwards
def dense_ff(h, w, pre, round_to):
    proj = lambda n, x: x @ w[pre + n].t() + w[pre + n + ".b"]
    return proj("down", _r(silu(_r(proj("gate", h), round_to)) * _r(proj("up", h), round_to), round_to))


def choose_experts(z, top: int, groups: Optional[Tuple[int, int]]):
    """z [T, E] router logits -> (chosen [T, top] best first, s [T, E], margin [T]).  s = sigmoid(z); with groups (count, keep)
    only members of the `keep` groups (neighbours, equal sizes) whose two best scores have the largest sum can be chosen.  The
    margin is how far rounding would have to move a logit to change the choice, to first order."""
    s = torch.sigmoid(z)
    T, E = s.shape
    margin = torch.full((T,), float("inf"))
    slope = s * (1.0 - s)                                                      # a logit moved by x moves a score by slope x
    c, allowed = s, torch.ones(T, E, dtype=torch.bool)
    if groups is not None and groups[1] < groups[0]:
        count, keep = groups
        two = torch.topk(s.view(T, count, -1), min(2, E // count), dim=-1)
        total = two.values.sum(-1)
        moves = slope.view(T, count, -1).gather(2, two.indices).sum(-1)
        order = torch.sort(total, dim=-1, descending=True).indices
        a, b = order[:, keep - 1:keep], order[:, keep:keep + 1]
        margin = ((total.gather(1, a) - total.gather(1, b)) / (moves.gather(1, a) + moves.gather(1, b)).clamp_min(1e-12))[:, 0].to(torch.float32)
        kept = torch.zeros(T, count, dtype=torch.bool).scatter_(1, order[:, :keep], True)
        allowed = kept.repeat_interleave(E // count, 1)
        c = s.masked_fill(~allowed, -1.0)
    order = torch.sort(c, dim=-1, descending=True).indices
    offered = allowed.sum(-1)
    if top < int(offered.min()):
        zz = z.gather(1, order[:, top - 1:top + 1])
        margin = torch.minimum(margin, ((zz[:, 0] - zz[:, 1]) / 2.0).to(torch.float32))
    return order[:, :top], s, margin


def routed_ff(h, w, pre, mlp, round_to, gaps=None):
    """scale * sum over the chosen of s_e / (sum of the chosen s + 1e-20) down_e gelu(up_e h), added in the order of the
    choices.  `gaps` (a list) receives the margins of the choices."""
    r, grp = mlp["router"], mlp["router"].get("groups")
    idx, s, margin = choose_experts(h @ w[pre + "router"].t(), r["top"], (grp["count"], grp["keep"]) if grp else None)
    if gaps is not None:
        gaps.append(margin)
    picked = s.gather(1, idx)
    weight = picked / (picked.sum(-1, keepdim=True) + 1e-20) * r["scale"]
    out = torch.zeros_like(h)
    for c in range(r["top"]):
        for e in idx[:, c].unique().tolist():
            rows = idx[:, c] == e
            y = _r(gelu_erf(h[rows] @ w[f"{pre}e{e}.up"].t()), round_to) @ w[f"{pre}e{e}.down"].t()
            out[rows] += weight[rows, c, None] * y
    return out


# --------------------------------------------------------------------- the arrangement of a layer
def gated(y, h, w, name, round_to):
    """A sublayer's result times sigmoid(W h + b), h being the sublayer's own input."""
    return y * torch.sigmoid(_r(h @ w[name].t(), round_to) + w[name + ".b"])


def read_streams(x, read):
    """x [T, S, D] -> sum_s read[s] x_s."""
    return torch.einsum("tsd,s->td", x, read)


def write_streams(x, mix, put, m, y):
    """x_b <- sum_a mix[a, b] x_a + m put[b] y, all streams from the old ones."""
    return torch.einsum("tad,ab->tbd", x, mix) + m * put[None, :, None] * y[:, None, :]


def runs(cfg) -> List[int]:
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


class PlainLopilix:
    def __init__(self, model_dir: str, round_to: Optional[torch.dtype] = None, wide: bool = False):
        with open(os.path.join(model_dir, "config.json")) as f:
            self.cfg = json.load(f)
        self.ft = torch.float64 if wide else torch.float32
        self.w: Dict[str, torch.Tensor] = {n: t.to(self.ft) for n, t in
                                           read_safetensors(os.path.join(model_dir, "model.safetensors")).items()}
        self.round_to = round_to
        self._gaps: list = []
        self.gaps = torch.zeros(0)

    def mixer(self, i: int, L: dict, h: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
        w, rt, eps, pre, m = self.w, self.round_to, self.cfg["norm"]["eps"], f"l{i}.mix.", L["mixer"]
        if L["type"] == "attention":
            heads = difference_attention(h, w, pre, m, eps, pos, rt)
        elif L["type"] == "hgrn2":
            heads = memory_mixer(h, w, pre, m, eps, calls=self._gaps)
        elif L["type"] == "latent_attention":
            heads = latent_attention(h, w, pre, m, eps, pos, rt)
        else:
            raise ValueError(L["type"])
        return _r(heads, rt) @ w[pre + "o"].t()

    def feed_forward(self, i: int, mlp: dict, h: torch.Tensor) -> torch.Tensor:
        if mlp["kind"] == "dense":
            return dense_ff(h, self.w, f"l{i}.mlp.", self.round_to)
        if mlp["kind"] == "moe":
            return routed_ff(h, self.w, f"l{i}.mlp.", mlp, self.round_to, self._gaps)
        raise ValueError(mlp["kind"])

    def sublayer(self, i: int, q: int, x: torch.Tensor, fn) -> torch.Tensor:
        """One sublayer of layer i (q 1: the mixer, 2: the feed-forward) on the streams x [T, S, D]."""
        w, hc = self.w, f"l{i}.hc{q}."
        h = self.norm(read_streams(x, w[hc + "in"]), f"l{i}.norm{q}")
        y = gated(fn(h), h, w, f"l{i}.rg{q}", self.round_to)
        return write_streams(x, w[hc + "mix"], w[hc + "out"], self.cfg["residual_mult"], y)

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return _r(unit_rms(x, self.cfg["norm"]["eps"]) * self.w[name], self.round_to)

    def forward(self, ids: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
        cfg = self.cfg
        pos = torch.arange(len(ids))
        self._gaps = []
        first = self.w["embed"][torch.tensor(list(ids), dtype=torch.long)] + self.w["pos"][:len(ids)]
        x = first[:, None, :].repeat(1, cfg["streams"], 1)
        for i in runs(cfg):
            L = cfg["layers"][i]
            x = self.sublayer(i, 1, x, lambda h: self.mixer(i, L, h, pos))
            if L.get("mlp") is not None:
                x = self.sublayer(i, 2, x, lambda h: self.feed_forward(i, L["mlp"], h))
            if layers_out is not None:
                layers_out.append(x.sum(1))
        # per position, the closest call any router or memory of the model made on it
        self.gaps = torch.stack(self._gaps).amin(0) if self._gaps else torch.full((len(ids),), float("inf"))
        return (self.norm(x.sum(1), "final.norm") @ self.w["embed"].t()) * cfg["logit_scale"]

    def logits(self, ids: Sequence[int]) -> torch.Tensor:
        return self.forward(ids).to(torch.float32)
