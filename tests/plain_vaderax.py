"""The plain implementation of the Vaderax design: whole sequences, no cache, no chunks, one function per mechanism,
elementary tensor arithmetic on the CPU; the delta rule runs token by token.

It shares no code with the engine: it reads config.json and model.safetensors itself.  `round_to` rounds to bfloat16
where the engine's bfloat16 path stores bfloat16 (the inputs of the matrix products, projections, cached rows); the
arithmetic itself is 32-bit (or 64-bit with `wide`).

Notation: D width, T tokens, H heads, G key/value heads, d query/key size per head, P value size per head, K taps of the
short convolution, E experts, I identity experts.
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
def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    """(x - mean) / sqrt(mean of (x - mean)^2 + eps) * w + b over the last axis."""
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_vector(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    """x / sqrt(sum(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) ** 2


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def rotate_half(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, d]: among the first `dims` coordinates of every head, coordinate i pairs with i + dims/2 and the pair
    (u, v) turns by the angle a = position * base^(-2i/dims): (u cos a - v sin a, v cos a + u sin a).  The rest pass."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64).to(torch.float32).to(x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def causal_conv(u: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """u [T, C], taps [C, K]: y_t = sum_j taps[:, j] u_(t - K + 1 + j), zeros before the start (the last column meets
    the present token)."""
    T, C = u.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=u.dtype), u], 0)
    y = torch.zeros(T, C, dtype=u.dtype)
    for j in range(K):
        y = y + padded[j:j + T] * taps[:, j]
    return y


# --------------------------------------------------------------------- mixers
def delta_rule(q, k, v, beta, keep, S=None, sizes=None):
    """q, k [T, H, d], v [T, H, P], beta and keep [T, H].  Per head: the memory decays, S <- keep S; what it answers to k is
    corrected towards v, u = beta (v - S^T k), S <- S + k u^T; then it is read, o = S^T q.  Returns o [T, H, P], S [H, d, P];
    `sizes` (a list) receives the norm of every head's S per token."""
    T, H, d = q.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = keep[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("adp,ad->ap", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("adp,ad->ap", S, q[t]))
        if sizes is not None:
            sizes.append(S.flatten(1).norm(dim=-1))
    return torch.stack(out), S


def delta_mixer(h, w, pre, m, eps, round_to, calls=None):
    """q, k (G heads) and v (H heads) pass a causal convolution and silu; q and k become unit vectors per head, q then times
    d^(-1/2); beta = sigmoid(W_b h), keep = exp(-exp(A_log) softplus(W_a h + dt_bias)); the delta rule, head a with the q and k
    of head a // (H / G); every head's o divided by its root mean square, times a weight shared by the heads, times silu(W_g h).
    Returns [T, H P].

    `calls` (a list) receives per token how far the model is from a close call: after the division by its root mean square only
    the direction of S^T q is left of a head's output, and where q is nearly orthogonal to what the memory holds (a memory of
    one token: the SIGN of k . q) rounding decides it.  2.5 sqrt(d) |S^T q| / (|S| |q|), the least over the heads."""
    H, G, d, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, rep = h.shape[0], m["heads"] // m["kv_heads"]
    mix = lambda n: silu(causal_conv(_r(h @ w[pre + n].t(), round_to), w[pre + n + ".conv"]))
    q = (unit_vector(mix("q").view(T, G, d)) * d ** -0.5).repeat_interleave(rep, 1)
    k = unit_vector(mix("k").view(T, G, d)).repeat_interleave(rep, 1)
    v = mix("v").view(T, H, P)
    beta = torch.sigmoid(h @ w[pre + "b"].t())
    keep = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].t() + w[pre + "dt_bias"]))
    sizes = None if calls is None else []
    o, _ = delta_rule(q, k, v, beta, keep, sizes=sizes)
    if calls is not None:
        hold = torch.stack(sizes) * q.norm(dim=-1)
        calls.append((2.5 * math.sqrt(d) * (o.norm(dim=-1) / hold.clamp_min(1e-30)).amin(-1)).to(torch.float32))
    o = (unit_rms(o, eps) * w[pre + "norm"]).reshape(T, H * P)
    return o * silu(_r(h @ w[pre + "g"].t(), round_to))


def attention(h, w, pre, m, eps, positions, round_to):
    """Grouped-query attention: the first rot.dims coordinates of every q and k head are rotated (rotate-half pairs), and each
    head is then divided by its root mean square; causal softmax over scale q . k; the heads, side by side, times
    sigmoid(W_g h).  Returns [T, H P]."""
    H, G, d, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T, rep = h.shape[0], m["heads"] // m["kv_heads"]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    proj = lambda n: _r(h @ w[pre + n].t(), round_to)
    q = _r(unit_rms(rotate_half(proj("q").view(T, H, d), positions, base, dims), eps), round_to)
    k = _r(unit_rms(rotate_half(proj("k").view(T, G, d), positions, base, dims), eps), round_to)
    kh, vh = k.repeat_interleave(rep, 1), proj("v").view(T, G, P).repeat_interleave(rep, 1)
    s = torch.einsum("iad,jad->aij", q, kh) * m["scale"]
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    p = e / e.sum(-1, keepdim=True)
    o = torch.einsum("aij,jad->iad", p, vh).reshape(T, H * P)
    return o * torch.sigmoid(proj("g"))


# --------------------------------------------------------------------- feed-forwards
def relu2_ff(h, w, pre, round_to):
    return _r(relu_squared(h @ w[pre + "up"].t()), round_to) @ w[pre + "down"].t()


def choose_experts(z, correction, top, groups: Optional[Tuple[int, int]]):
    """z [T, E + I] router logits -> (chosen [T, top] best first, their scores [T, top], margin [T]).  s = softmax(z); the
    choice goes by s + correction; with groups (count, keep) only members of the `keep` groups (neighbours, equal sizes) whose
    largest choice score is largest can be chosen.  The margin is how far rounding would have to move a choice score to change
    the choice, in units of the score at the boundary (a change of a logit by x moves a score by about that factor)."""
    s = torch.softmax(z, -1)
    c = s + correction
    T, N = c.shape
    margin = torch.full((T,), float("inf"))

    def gap(values, scores_at, last):
        """Distance between place `last` and the next one of sorted `values`, over the sum of both places' softmax scores."""
        order = torch.sort(values, dim=-1, descending=True)
        a, b = order.values[:, last - 1], order.values[:, last]
        sa = scores_at.gather(1, order.indices[:, last - 1:last])[:, 0]
        sb = scores_at.gather(1, order.indices[:, last:last + 1])[:, 0]
        return ((a - b) / (sa + sb).clamp_min(1e-12)).to(torch.float32)
    if groups is not None and groups[1] < groups[0]:
        count, keep = groups
        by_group = c.view(T, count, N // count)
        best, where = by_group.max(-1)
        kept = torch.topk(best, keep, dim=-1).indices
        margin = torch.minimum(margin, gap(best, s.view(T, count, -1).gather(2, where[..., None])[..., 0], keep))
        allowed = torch.zeros(T, count, dtype=torch.bool).scatter_(1, kept, True)
        c = by_group.masked_fill(~allowed[..., None], float("-inf")).reshape(T, N)
    idx = torch.topk(c, top, dim=-1).indices
    if top < N:
        g = gap(c, s, top)
        margin = torch.minimum(margin, torch.where(torch.isnan(g), torch.full_like(g, float("inf")), g))
    return idx, s.gather(1, idx), margin


def routed_ff(h, w, pre, mlp, round_to, gaps=None):
    """The chosen experts' outputs times their softmax scores (not renormalised), added in the order of the choices; the last I
    of the E + I router outputs stand for the input itself.  `gaps` (a list) receives the margins of the choices."""
    r = mlp["router"]
    E, I = r["experts"], r.get("identity") or 0
    z = h @ w[pre + "router"].t()
    grp = r.get("groups")
    idx, s, margin = choose_experts(z, w[pre + "correction"], r["top"], (grp["count"], grp["keep"]) if grp else None)
    if gaps is not None:
        gaps.append(margin)
    out = torch.zeros_like(h)
    for c in range(r["top"]):
        for e in idx[:, c].unique().tolist():
            rows = idx[:, c] == e
            y = relu2_ff(h[rows], w, f"{pre}e{e}.", round_to) if e < E else h[rows]
            out[rows] += s[rows, c, None] * y
    return out


# --------------------------------------------------------------------- the model
def runs(cfg) -> List[Tuple[int, bool]]:
    """The layers in the order they run, each with whether the embedding output is added to x right before it."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, p > 0 and i == a) for p in range(loop["times"]) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body + [(i, False) for i in range(b, n)]


class PlainVaderax:
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
        w, rt, eps, pre = self.w, self.round_to, self.cfg["norm"]["eps"], f"l{i}.mix."
        if L["type"] == "delta":
            heads = delta_mixer(h, w, pre, L["mixer"], eps, rt, calls=self._gaps)
        elif L["type"] == "attention":
            heads = attention(h, w, pre, L["mixer"], eps, pos, rt)
        else:
            raise ValueError(L["type"])
        return _r(heads, rt) @ w[pre + "o"].t()

    def feed_forward(self, i: int, mlp: dict, h: torch.Tensor) -> torch.Tensor:
        if mlp["kind"] == "dense":
            return relu2_ff(h, self.w, f"l{i}.mlp.", self.round_to)
        if mlp["kind"] == "moe":
            return routed_ff(h, self.w, f"l{i}.mlp.", mlp, self.round_to, self._gaps)
        raise ValueError(mlp["kind"])

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return _r(layer_norm(x, self.w[name], self.w[name + ".b"], self.cfg["norm"]["eps"]), self.round_to)

    def forward(self, ids: Sequence[int], layers_out: Optional[list] = None) -> torch.Tensor:
        cfg = self.cfg
        pos = torch.arange(len(ids))
        self._gaps = []
        first = self.w["embed"][torch.tensor(list(ids), dtype=torch.long)] * float(cfg["embedding"]["scale"])
        x = first.clone()
        for i, again in runs(cfg):
            L = cfg["layers"][i]
            if again:
                x = x + first
            x = x + self.mixer(i, L, self.norm(x, f"l{i}.norm1"), pos)
            if L.get("mlp") is not None:
                x = x + self.feed_forward(i, L["mlp"], self.norm(x, f"l{i}.norm2"))
            if layers_out is not None:
                layers_out.append(x.clone())
        # per position, the closest call any router or memory of the model made on it
        self.gaps = torch.stack(self._gaps).amin(0) if self._gaps else torch.full((len(ids),), float("inf"))
        return self.norm(x, "final.norm") @ self.w["head"].t()

    def logits(self, ids: Sequence[int]) -> torch.Tensor:
        return self.forward(ids).to(torch.float32)
