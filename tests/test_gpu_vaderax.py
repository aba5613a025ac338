"""The Vaderax design on the GPU against the plain implementation: single kernels, each mixer in a model of its own, every
schedule in both precisions and with both kernel sets, constants that are one off (negative controls on the plain
implementation, then the engine with the right ones), a key far back that stands out, a first token that only the memory
remembers, decoding from the first token on through captured steps, generation through the scheduler, the trace program."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

from helpers import compare, engine_for, max_live_tokens, random_ids, replay, trace_bulk_then_single, trace_portions, trace_whole
from plain_vaderax import PlainVaderax, choose_experts, delta_rule, layer_norm, relu_squared, silu, softplus, unit_rms, unit_vector
from test_gpu_vifelix import _batch, _ops, _run
from tiny_vaderax import (ONE_PASS, ONLY_ATTENTION, ONLY_DELTA, TINY_A, TINY_B, attention, delta, dense, layer, make_vaderax_dir, model, moe)
from vaderax_cases import greedy_by_the_plain_model, reference_logits, replay_all_schedules, schedules, variant_dir

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"


# ----------------------------------------------------------------------------- single kernels
def _step_spans(lens, cuts, step):
    """Which tokens of which request a step brings, when every request is cut in two at a place of its own."""
    spans = [(r, 0, cuts[r]) if step == 0 else (r, cuts[r], lens[r]) for r in range(len(lens))]
    return [s for s in spans if s[2] > s[1]]


@pytest.mark.parametrize("kernels", ["fast", "plain"])
@pytest.mark.parametrize("H,G,n,p", [(1, 1, 4, 3), (4, 2, 8, 16), (3, 1, 6, 5), (2, 2, 32, 48), (6, 2, 64, 33), (4, 1, 128, 20), (2, 1, 100, 64),
                                     (2, 2, 200, 9), (1, 1, 500, 6), (40, 4, 12, 24), (24, 12, 60, 70), (48, 8, 128, 17)])
def test_delta_rule_kernels(H, G, n, p, kernels):
    """Single tokens beside portions (down to two tokens, no multiples of four, hundreds) in slots that are not in order; the second
    step starts every request from the state the first one left.  Keys come again (the write replaces what the memory holds), write
    strengths reach 0 and 1 and decays 0 and 1."""
    ops = _ops(kernels)
    g = torch.Generator().manual_seed(n + p)
    lens, cuts, slots = [331, 1, 128, 65, 2, 9], [200, 0, 63, 0, 1, 7], [1, 3, 0, 5, 2, 7]
    mk = lambda *s: torch.randn(*s, generator=g)
    q, k, v = [mk(L, G * n) for L in lens], [mk(L, G * n) for L in lens], [mk(L, H * p) for L in lens]
    gates = [torch.cat([2 * mk(L, H), 2 * mk(L, H)], 1) for L in lens]
    for r, L in enumerate(lens):
        for t in range(3, L, 5):
            k[r][t] = k[r][t - 2]
        gates[r][L // 3::17, :H] = 80.0
        gates[r][L // 4::23, :H] = -80.0
        gates[r][L // 5::29, H:] = 300.0             # a decay of zero: the memory is emptied
        gates[r][L // 2::13, H:] = -80.0
    a_log, dt_bias = mk(H) - 1.0, mk(H) - 2.0
    state = torch.zeros(max(slots) + 2, H, p, n, device=DEV)
    T = sum(lens)
    unit = torch.full((T, 2 * G * ((n + 3) // 4 * 4)), float("nan"), device=DEV)
    coef = torch.full(((T // 8 + len(lens) + 1) * H * 160,), float("nan"), device=DEV)
    got = [[] for _ in lens]
    for step in range(2):
        spans = _step_spans(lens, cuts, step)
        cat = lambda xs: torch.cat([xs[r][a:b] for r, a, b in spans]).to(DEV)
        gt = cat(gates)
        out = torch.zeros(gt.shape[0], H * p, device=DEV)
        _run(ops, lambda pl: pl.delta_rule(q=cat(q), k=cat(k), v=cat(v), write=gt[:, :H], forget=gt[:, H:], dt_bias=dt_bias.to(DEV),
                                           a_log=a_log.to(DEV), q_scale=n ** -0.5, unit_eps=1e-6, state=state, out=out, heads=H, n=n, p=p,
                                           qk_groups=G, unit=unit, coef=coef),
             _batch([b - a for _, a, b in spans], [slots[r] for r, _, _ in spans]))
        at = 0
        for r, a, b in spans:
            got[r].append(out[at:at + b - a].cpu())
            at += b - a
    for r, L in enumerate(lens):
        heads = lambda x: x.view(L, G, n).double().repeat_interleave(H // G, 1)
        beta = torch.sigmoid(gates[r][:, :H].double())
        keep = torch.exp(-torch.exp(a_log.double()) * softplus(gates[r][:, H:].double() + dt_bias.double()))
        want, S = delta_rule(unit_vector(heads(q[r])) * n ** -0.5, unit_vector(heads(k[r])), v[r].view(L, H, p).double(), beta, keep)
        y = torch.cat(got[r]).view(L, H, p)
        assert float((y - want).abs().max()) < 2e-5 * max(1.0, float(want.abs().max())), r
        assert float((state[slots[r]].cpu() - S.transpose(1, 2)).abs().max()) < 2e-5 * max(1.0, float(S.abs().max())), r
    assert float(state[max(slots) + 1].abs().max()) == 0.0 and float(state[4].abs().max()) == 0.0


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("D", [20, 64, 1100, 2050, 4096])
def test_layer_norm_kernel(dtype, tol, D):
    """A mean far from zero, the pending addition in the same pass, all rows and only the wanted ones."""
    from llmengine_b200.engine.batch import StepBatch
    ops = _ops()
    g = torch.Generator().manual_seed(D)
    T = 7
    x, add = torch.randn(T, D, generator=g) + 30.0, torch.randn(T, D, generator=g)
    w, b = (1 + 0.2 * torch.randn(D, generator=g)).to(dtype), torch.randn(D, generator=g).to(dtype)
    xd, out = x.to(DEV), torch.zeros(T + 1, D, dtype=dtype, device=DEV)
    full = lambda t: torch.cat([t, torch.zeros(1, D, device=DEV)])
    xs, adds = full(xd), full(add.to(DEV))
    _run(ops, lambda p: p.layernorm(xs, w.to(DEV), b.to(DEV), 1e-5, out, delta=adds), _batch([T], [0]))
    want = layer_norm((x + add).double(), w.double(), b.double(), 1e-5)
    assert float((out[:T].double().cpu() - want).abs().max()) < tol * 3 and float(out[T].abs().max()) == 0.0
    assert float((xs[:T].cpu() - (x + add)).abs().max()) < 1e-5
    rows = torch.tensor([5, 0, 3], dtype=torch.int32, device=DEV)
    got = torch.zeros(T, D, dtype=dtype, device=DEV)
    _run(ops, lambda p: p.layernorm(xs, w.to(DEV), b.to(DEV), 1e-5, got, rows="logits"),
         StepBatch.bare(T, torch.device(DEV), logit_rows=rows, logits=torch.zeros(3, 4, device=DEV)))
    assert float((got[:3].double().cpu() - want[[5, 0, 3]]).abs().max()) < tol * 3


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
def test_small_records_of_the_design(dtype, tol):
    """The embedding output added to a stream that exists; the square of relu behind a product (few tokens, many, and shapes that
    no tensor-core product takes); the gated norm with a 32-bit gate."""
    ops = _ops()
    g = torch.Generator().manual_seed(5)
    for D in (24, 300, 1040):
        table = torch.randn(11, D, generator=g).to(dtype)
        x, add, ids = torch.randn(6, D, generator=g), torch.randn(6, D, generator=g), [3, 10, 0, 0, 7, 5]
        b = _batch([6], [0])
        b.token_ids.copy_(torch.tensor(ids, dtype=torch.int32))
        for pending in (None, add.to(DEV)):
            xd = x.to(DEV)
            _run(ops, lambda p: p.embedding(table.to(DEV), xd, scale=2.5, accumulate=True, delta=pending), b)
            want = x + (add if pending is not None else 0.0) + table[ids].float() * 2.5
            assert float((xd.cpu() - want).abs().max()) < 1e-5
    for T, K, N in ((3, 40, 24), (16, 264, 130), (200, 128, 520), (300, 36, 20)):
        x, w = torch.randn(T, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) / math.sqrt(K)).to(dtype)
        mid, out = torch.zeros(T, N, dtype=dtype, device=DEV), torch.zeros(T, N, dtype=dtype, device=DEV)
        for choice in ({}, {"linear": "tcgen05", "linear.decode": "skinny"}, {"linear": "plain"}):
            o = _ops(choice or "fast")
            _run(o, lambda p: p.linear_act(x.to(DEV), w.to(DEV), mid, out, "relu2"), _batch([T], [0]))
            assert float((out.float().cpu() - relu_squared(x.float() @ w.float().t())).abs().max()) < tol * 4, (T, choice)
    for groups, group in ((3, 5), (4, 32), (2, 300)):
        T, cols = 7, groups * group
        y, gate, w = torch.randn(T, cols, generator=g) * 3, torch.randn(T, cols + 2, generator=g), 1 + 0.2 * torch.randn(cols, generator=g)
        gd, out = gate.to(DEV), torch.zeros(T + 1, cols, dtype=dtype, device=DEV)
        _run(ops, lambda p: p.gated_norm(y=y.to(DEV), gate=gd[:, 1:1 + cols], weight=w.to(DEV), out=out, group=group, gate_first=False, eps=1e-5),
             _batch([T], [0]))
        want = unit_rms(y.view(T, groups, group), 1e-5).reshape(T, cols) * w * silu(gate[:, 1:1 + cols])
        assert float((out[:T].float().cpu() - want).abs().max()) < tol * max(1.0, float(want.abs().max())) and float(out[T].abs().max()) == 0.0


@pytest.mark.parametrize("T", [5, 64, 65, 200])
@pytest.mark.parametrize("E,I,top,groups", [(5, 0, 1, (1, 1)), (7, 2, 3, (3, 2)), (12, 0, 3, (4, 1)), (3, 1, 4, (2, 2)), (60, 4, 9, (8, 3)), (130, 20, 6, (5, 2))])
def test_routing_by_the_softmax_over_all(E, I, top, groups, T):
    """The corrected scores choose, inside the best groups only; the weights are the scores themselves; pairs are listed expert by
    expert; in the weighted sum the identity experts stand for the input."""
    ops = _ops()
    g = torch.Generator().manual_seed(E + T)
    N, D = E + I, 12
    wide, corr = (torch.randn(T, N + 3, generator=g) * 1.5).to(DEV), 0.3 * torch.randn(N, generator=g) - 0.2
    experts, weights = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
    offsets, counts = torch.zeros(N + 1, dtype=torch.int32, device=DEV), torch.zeros(N, dtype=torch.int32, device=DEV)
    order = torch.zeros(T * top, dtype=torch.int32, device=DEV)
    y, h, out = torch.randn(T * top, D, generator=g), torch.randn(T, D, generator=g), torch.zeros(T, D, device=DEV)
    idx, wt, margin = choose_experts(wide[:, :N].cpu(), corr, top, groups)
    clear = margin > 1e-4                          # (positions where rounding decides prove nothing)
    assert int(clear.sum()) > 0.8 * T
    y[(idx.reshape(-1) >= E).nonzero()[:, 0]] = float("nan")           # rows that no product writes
    hd = h.to(DEV)

    def records(p):
        p.moe_route(logits=wide[:, :N], top_k=top, scale=1.0, experts=experts, weights=weights, offsets=offsets, order=order, counts=counts,
                    mode="softmax", correction=corr.to(DEV), groups=groups)
        p.moe_combine(y=y.to(DEV), weights=weights, base=None, out=out, experts=experts if I else None, identity=hd if I else None, first_identity=E)
    for _ in range(2):                             # (the second launch finds the counters as it needs them)
        _run(ops, records, _batch([T], [0]))
    assert torch.equal(experts.cpu().long()[clear], idx[clear])
    assert float((weights.cpu() - wt)[clear].abs().max()) < 1e-6
    off, od, ex = offsets.cpu().tolist(), order.cpu().tolist(), experts.cpu().reshape(-1).tolist()
    for e in range(N):
        assert sorted(od[off[e]:off[e + 1]]) == [i for i in range(T * top) if ex[i] == e]
    rows = torch.where((idx >= E)[:, :, None], h[:, None, :], y.view(T, top, D))
    want = (wt[:, :, None] * rows).sum(1)
    assert float((out.cpu() - want)[clear].abs().max()) < 1e-5 and float(counts.abs().max()) == 0


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("kernels", ["fast", "tcgen05", "mma"])
@pytest.mark.parametrize("T,E,top,n,k", [(3, 5, 2, 24, 40), (150, 4, 3, 72, 64), (40, 3, 1, 20, 36), (300, 6, 4, 264, 192), (700, 2, 2, 520, 328)])
def test_grouped_products_with_the_square_of_relu(dtype, tol, T, E, top, n, k, kernels):
    """Both products of ungated experts: gathered by token with the square of relu in the epilogue, scattered by pair; the pairs of
    identity experts (behind the experts' in the order) are no product's.  Experts of no row, of a few and of several tiles."""
    ops = _ops(kernels if kernels == "fast" else {"grouped_linear": kernels})
    g = torch.Generator().manual_seed(T)
    choice = torch.stack([torch.randperm(E + 1, generator=g)[:top] for _ in range(T)])
    order = torch.argsort(choice.reshape(-1), stable=True)
    offsets = torch.cat([torch.zeros(1, dtype=torch.long), torch.cumsum(torch.bincount(choice.reshape(-1), minlength=E + 1), 0)])
    x, up, down = torch.randn(T, k, generator=g).to(dtype), (torch.randn(E, n, k, generator=g) / math.sqrt(k)).to(dtype), \
        (torch.randn(E, k, n, generator=g) / math.sqrt(n)).to(dtype)
    act, mid = torch.zeros(T * top, n, dtype=dtype, device=DEV), torch.zeros(T * top, n, dtype=dtype, device=DEV)
    y = torch.full((T * top, k), float("nan"), device=DEV)
    lists = dict(offsets=offsets.to(torch.int32).to(DEV), order=order.to(torch.int32).to(DEV), top_k=top)

    rows = torch.zeros(T * top, k, dtype=dtype, device=DEV)

    def records(p):
        p.grouped_linear(x=x.to(DEV), w=up.to(DEV), out=act, gather=True, scatter=False, mid=mid, act="relu2", rows=rows, **lists)
        p.grouped_linear(x=act, w=down.to(DEV), out=y, gather=False, scatter=True, **lists)
    _run(ops, records, _batch([T], [0]))
    if "moe_tcgen05" in ops._libs:
        assert ops.grouped_tcgen05_status() == 0
    for i, e in enumerate(choice.reshape(-1).tolist()):
        row = y[i].cpu()
        if e == E:
            assert torch.isnan(row).all()
            continue
        a = relu_squared(up[e].float() @ x[i // top].float()).to(dtype).float()
        assert float((row - down[e].float() @ a).abs().max()) < tol * 3, (i, e)


@pytest.mark.parametrize("out_dtype", [torch.bfloat16, torch.float32])
def test_gated_grouped_product_on_tcgen05(out_dtype):
    """The same kernel with silu(gate) up in its epilogue, against the warp-level kernel, for experts of 0, 1, 128, 129 and more rows."""
    g = torch.Generator().manual_seed(8)
    E, n, k, rows = 6, 328, 136, [0, 1, 128, 129, 300, 7]
    order = torch.randperm(sum(rows), generator=g)
    offsets = torch.tensor([0] + list(np.cumsum(rows)))
    x, w = torch.randn(sum(rows), k, generator=g).to(torch.bfloat16).to(DEV), (torch.randn(E, 2 * n, k, generator=g) / 12).to(torch.bfloat16).to(DEV)
    outs = []
    for how in ("tcgen05", "mma"):
        ops = _ops({"grouped_linear": how})
        out, place = torch.full((sum(rows) + 1, n), 7.0, dtype=out_dtype, device=DEV), torch.zeros(sum(rows), k, dtype=torch.bfloat16, device=DEV)
        _run(ops, lambda p: p.grouped_linear(x=x, w=w, out=out, offsets=offsets.to(torch.int32).to(DEV), order=order.to(torch.int32).to(DEV), top_k=1,
                                             gather=True, scatter=True, act="silu", rows=place), _batch([sum(rows)], [0]))
        outs.append(out.float().cpu())
    assert float((outs[0] - outs[1]).abs().max()) < 2e-2 * max(1.0, float(outs[1].abs().max())) and float((outs[0][-1] - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("taps", [2, 4, 5])
def test_convolution_of_single_tokens_in_one_launch(taps):
    """A step in which every request brings one token: the outputs and the stored inputs of one launch are those of the two that
    serve other steps."""
    ops = _ops()
    g = torch.Generator().manual_seed(taps)
    C, R = 90, 3
    w, b = torch.randn(C, taps, generator=g), torch.randn(C, generator=g)
    state = torch.zeros(5, taps - 1, C, device=DEV)
    xs = torch.randn(2 * taps + 1, R, C, generator=g)
    slots = [4, 0, 2]
    for x in xs:
        out = torch.zeros(R, C, device=DEV)
        _run(ops, lambda p: p.short_conv(x=x.to(DEV), w=w.to(DEV), bias=b.to(DEV), state=state, out=out, act="silu"), _batch([1] * R, slots))
        last = out.cpu()
    for r in range(R):
        want = silu(b + sum(w[:, taps - 1 - j] * xs[-1 - j, r] for j in range(taps)))
        assert float((last[r] - want).abs().max()) < 1e-5
        assert torch.equal(state[slots[r]].cpu(), xs[-(taps - 1):, r])
    assert float(state[1].abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


# ----------------------------------------------------------------------------- each mixer in a model of its own
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg", [("delta", ONLY_DELTA), ("attention", ONLY_ATTENTION), ("one pass", ONE_PASS)])
def test_each_mixer_alone(tmp_path, name, cfg, dtype):
    d = make_vaderax_dir(str(tmp_path / "m"), cfg, seed=9)
    replay_all_schedules(d, cfg, dtype, [70, 5, 130, 1, 2], 16, None, DEV, only=("whole", "bulk_then_single", "portions"))


# ----------------------------------------------------------------------------- every schedule
# sizes the tensor-core kernels take: heads of 64 (the tcgen05 portion kernel), of 48 and of 80 with values of 32, states of 64 and 128
# rows, experts in whole tiles
BIG = model(131, 128, 1e-6, 9.0, [
    layer("attention", attention(4, 2, 64, 64, 0.125, base=5000.0, dims=32), moe(6, 2, 64, identity=2, groups=(2, 1))),
    layer("delta", delta(4, 2, 64, 32, 4), dense(192)),
    layer("delta", delta(2, 1, 128, 64, 3), dense(96)),
    layer("attention", attention(6, 2, 48, 48, 0.2, base=300.0)),
    layer("attention", attention(2, 1, 80, 32, 0.2, base=100.0, dims=20), dense(160)),
], loop=(1, 3, 2))


@pytest.mark.parametrize("kernels", ["fast", "plain"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg,page,lens", [
    ("A", TINY_A, 16, [70, 33, 50, 1, 19, 64]),
    ("B", TINY_B, 8, [2, 5, 64, 90, 48]),
    ("D", ONLY_DELTA, 64, [150, 3, 40, 64, 7]),
    ("BIG", BIG, 64, [150, 40, 129, 2, 64]),
    ("BIG16", BIG, 16, [150, 40, 129, 2, 64]),
])
def test_replay_gpu(tmp_path, name, cfg, page, lens, dtype, kernels):
    d = make_vaderax_dir(str(tmp_path / name), cfg, seed=11)
    worst = replay_all_schedules(d, cfg, dtype, lens, page, None, DEV, kernels=kernels)
    print(f"replay {name} {dtype} {kernels}: share of the tolerance: " + ", ".join(f"{k} {v:.2f}" for k, v in worst.items()))


def test_replay_with_the_experts_products_on_tcgen05(tmp_path):
    """Every step's experts through the kernel that otherwise serves long prompts alone: tiles of a few rows, rows that run on into
    the next expert's."""
    d = make_vaderax_dir(str(tmp_path / "m"), BIG, seed=11)
    replay_all_schedules(d, BIG, "bfloat16", [150, 40, 129, 2, 64], 64, None, DEV, kernels={"grouped_linear": "tcgen05"})


# ----------------------------------------------------------------------------- constants that are one off
EDGE = model(50, 64, 1e-5, 6.0, [
    layer("attention", attention(4, 2, 32, 32, 0.2, base=200.0, dims=8), moe(6, 3, 32, identity=2, groups=(4, 2))),
    layer("delta", delta(2, 1, 16, 16, 3), dense(48)),
], loop=(0, 2, 2))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_constants_that_are_one_off(tmp_path, dtype):
    """Other rotated coordinates, another base or scale, one expert fewer, more groups kept, an identity expert counted as none,
    another number of passes, a loop over other layers, an embedding that is not scaled: each moves the plain implementation's logits
    far beyond the tolerance.  The engine, with the right constants, stays within it at every position, in prompts and decoded."""
    d = make_vaderax_dir(str(tmp_path / "edge"), EDGE, seed=31)
    reqs = {"a": random_ids(90, 50, 1), "b": random_ids(23, 50, 2), "c": random_ids(5, 50, 3)}
    ref, tol = reference_logits(d, reqs, dtype)
    router = lambda c: c["layers"][0]["mlp"]["router"]
    changes = {
        "more coordinates rotated": lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 10),
        "another base": lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("base", 4.0),
        "another scale": lambda c: c["layers"][0]["mixer"].__setitem__("scale", 0.8),
        "one expert per token": lambda c: router(c).__setitem__("top", 1),
        "three groups kept": lambda c: router(c)["groups"].__setitem__("keep", 3),
        "groups of four": lambda c: router(c).__setitem__("groups", {"count": 2, "keep": 1}),
        "no groups": lambda c: router(c).pop("groups"),
        "one more pass": lambda c: c["loop"].__setitem__("times", 3),
        "no loop": lambda c: c.pop("loop"),
        "a loop over one layer": lambda c: c["loop"].__setitem__("start", 1),
        "embedding not scaled": lambda c: c["embedding"].__setitem__("scale", 1.0),
        "another eps": lambda c: c["norm"].__setitem__("eps", 0.3),
    }
    for what, change in changes.items():
        other = PlainVaderax(variant_dir(d, str(tmp_path / what.replace(" ", "_")), change))
        moved = float((other.logits(reqs["a"]) - ref["a"]).abs().max())
        assert moved > 3 * tol, f"{what} moves the logits by {moved:.3g} only (tolerance {tol:.3g})"
    for page in (4, 16, 64):
        for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_bulk_then_single(reqs, 60)), ("portions", trace_portions(reqs))):
            eng = engine_for(d, dtype, 256, page_size=page, max_requests=2, max_model_len=128)
            compare(replay(eng, steps, poison=True), ref, tol, f"{dtype}/page {page}/{what}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dk", [16, 64])
def test_a_key_far_back_among_hundreds(tmp_path, dtype, dk):
    """One token's key points along a coordinate that is not rotated, and every query points there too.  Put at position 3 of 400 it
    still takes most of the attention at the end, over page borders: exchanging it moves the last logits by many tolerances, in
    the plain implementation and, within the tolerance of it, in the engine."""
    H, G = 4, 2
    cfg = model(40, 48, 1e-5, 4.0, [layer("attention", attention(H, G, dk, dk, 14.0 / dk, base=100.0, dims=8), dense(24))])

    def change(w):
        e = w["embed"].float()
        e[:, 0] = 0.5                                 # a part of every input that does not depend on the token
        w["embed"] = e.to(torch.bfloat16)
        h7 = layer_norm(w["embed"][7].float() * 4.0, w["l0.norm1"].float(), w["l0.norm1.b"].float(), 1e-5)
        others = layer_norm(w["embed"].float() * 4.0, w["l0.norm1"].float(), w["l0.norm1.b"].float(), 1e-5)
        probe = torch.linalg.lstsq(others, torch.nn.functional.one_hot(torch.tensor(7), 40).float()[:, None]).solution[:, 0]
        probe = probe / (probe @ h7)                  # large on token 7 alone
        q, k = w["l0.mix.q"].float() * 0.3, w["l0.mix.k"].float() * 0.5
        for b in range(G):
            k[(b + 1) * dk - 1] = 6.0 * probe
        for a in range(H):
            q[(a + 1) * dk - 1] = 0.0
            q[(a + 1) * dk - 1, 0] = 4.0
        g = w["l0.norm1"].float()
        g[0] = 1.0
        w.update({"l0.mix.k": k.to(torch.bfloat16), "l0.mix.q": q.to(torch.bfloat16), "l0.norm1": g.to(torch.bfloat16)})
    d_ = make_vaderax_dir(str(tmp_path / "m"), cfg, seed=3, change=change)
    ids = [t if t != 7 else 8 for t in random_ids(400, 40, 5)]
    ids[3] = 7
    reqs = {"a": ids, "b": ids[:70]}
    ref, tol = reference_logits(d_, reqs, dtype)
    without = list(ids)
    without[3] = 9
    plain = PlainVaderax(d_)
    moved = float((plain.logits(ids)[-1] - plain.logits(without)[-1]).abs().max())
    assert moved > 10 * tol, f"the far token moves the logits by {moved:.3g} (tolerance {tol:.3g})"
    for page in (16, 64):
        for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_bulk_then_single(reqs, 40)), ("portions", trace_portions(reqs))):
            eng = engine_for(d_, dtype, 512, page_size=page, max_requests=2, max_model_len=512)
            compare(replay(eng, steps, poison=True), ref, tol, f"{dtype}/page {page}/{what}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_first_token_that_only_the_memory_remembers(tmp_path, dtype):
    """Delta layers alone, decays near one and small write strengths, in a loop whose every pass has a state of its own: changing the
    FIRST token of a prompt of 200 still moves the last logits, so a state that is lost, zeroed, shared between passes or taken from
    another slot on the way (portions, single tokens, slots used again) would show there."""
    cfg = model(45, 48, 1e-5, 5.0, [
        layer("delta", delta(4, 2, 32, 16, 2), dense(40)),
        layer("delta", delta(3, 3, 40, 16, 3)),
    ], loop=(0, 1, 2))

    def change(w):
        for i in (0, 1):
            w[f"l{i}.mix.dt_bias"] = torch.full_like(w[f"l{i}.mix.dt_bias"], -9.0)        # log decays about -1e-4
            w[f"l{i}.mix.b"] = w[f"l{i}.mix.b"] * 0.3
    d = make_vaderax_dir(str(tmp_path / "m"), cfg, seed=6, change=change)
    reqs = {f"r{i}": random_ids(n, 45, 70 + i) for i, n in enumerate([200, 40, 170, 9, 130])}
    ref, tol = reference_logits(d, reqs, dtype)
    plain = PlainVaderax(d)
    other = list(reqs["r0"])
    other[0] = (other[0] + 1) % 45
    if dtype == "float32":      # bfloat16 rounding of hundreds of tokens' writes moves these logits more than the first token does
        assert float((plain.logits(other)[-1] - ref["r0"][-1]).abs().max()) > 5 * tol
    for what, steps in schedules(reqs, tail=40).items():
        eng = engine_for(d, dtype, max_live_tokens(steps, 64), page_size=16, max_requests=4, max_model_len=512)
        compare(replay(eng, steps, poison=True), ref, tol, f"far/{dtype}/{what}")


# ----------------------------------------------------------------------------- from the first token on, for long
@pytest.mark.parametrize("cfg_name", ["A", "D"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoding_from_the_first_token_through_captured_steps(tmp_path, dtype, cfg_name):
    """Three requests decoded token by token from position 0 on, over several pages, with the steps captured in CUDA graphs: the same
    logits as whole prompts.  Also for a model that keeps no pages at all."""
    from llmengine_b200.engine.engine import StepEntry
    cfg = TINY_A if cfg_name == "A" else ONLY_DELTA
    d = make_vaderax_dir(str(tmp_path / "m"), cfg, seed=13)
    n = 70
    reqs = {f"r{i}": random_ids(n, cfg["vocab"], 50 + i) for i in range(3)}
    ref, tol = reference_logits(d, reqs, dtype)
    eng = engine_for(d, dtype, 3 * 192, page_size=16, max_requests=4, use_cuda_graphs=True, max_model_len=192)
    rows = {r: [] for r in reqs}
    for i in range(n):
        out = eng.step([StepEntry(r, [ids[i]], [0]) for r, ids in reqs.items()], list(reqs) if i == n - 1 else [])
        for k, r in enumerate(reqs):
            rows[r].append(out[k].float().cpu().clone())
    assert eng.graphs_enabled and eng._graphs, "the parts of this design can be captured"
    compare({r: torch.stack(v) for r, v in rows.items()}, ref, tol, f"captured decode {dtype}")
    eng.cache.check_invariants()
    assert all(g.pool.free_count == g.pool.num_pages for g in eng.cache.groups)


def test_greedy_generation_through_the_scheduler(tmp_path):
    from llmengine_b200 import LLM, SamplingParams
    d = make_vaderax_dir(str(tmp_path / "m"), TINY_A, seed=5)
    llm = LLM(d, dtype="float32", page_size=16, max_cached_tokens=512, max_num_seqs=4, max_num_batched_tokens=64,
              prefill_chunk=40, max_model_len=256)
    prompts = [random_ids(n, TINY_A["vocab"], i) for i, n in enumerate([1, 5, 64, 90, 33, 7])]
    outs = llm.generate(prompts, SamplingParams(greedy=True), max_tokens=12, eos_token_id=None)
    plain = PlainVaderax(d)
    for p, o in zip(prompts, outs):
        assert o.token_ids == greedy_by_the_plain_model(plain, p, 12)
    llm.engine.cache.check_invariants()
    assert not llm.engine.cache.requests and llm.scheduler.all_done()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(tmp_path, dtype):
    cfg = TINY_A
    d = make_vaderax_dir(str(tmp_path / "m"), cfg, seed=17)
    reqs = {f"r{i}": random_ids(n, cfg["vocab"], 200 + i) for i, n in enumerate([40, 33, 60, 1, 19, 25])}
    ref, tol = reference_logits(d, reqs, dtype)
    steps = schedules(reqs)["mixed"]
    out = tmp_path / "out"
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in e], "end": end})
             for i, (e, end) in enumerate(steps)]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out", str(out),
                        "--max-tokens", str(max_live_tokens(steps, 64))],
                       input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    rows = {}
    for i, (e, _) in enumerate(steps):
        arr = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        k = 0
        for r, t, w in e:
            rows.setdefault(r, []).append(arr[k:k + len(w)])
            k += len(w)
        assert k == arr.shape[0]
    compare({r: torch.cat(v) for r, v in rows.items()}, ref, tol, f"trace_run/{dtype}")
