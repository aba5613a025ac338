"""The Lopilix design on the GPU against the plain implementation: single kernels, each mixer in a model of its own, every
schedule in both precisions and with both kernel sets, constants that are one off (negative controls on the plain
implementation, then the engine with the right ones), keys far back that stand out, a first token that only the memory
remembers, decoding from the first token on through captured steps, generation through the scheduler, the trace program."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

from helpers import compare, engine_for, max_live_tokens, random_ids, replay, trace_bulk_then_single, trace_portions, trace_whole
from lopilix_cases import greedy_by_the_plain_model, reference_logits, replay_all_schedules, schedules, variant_dir
from plain_lopilix import (PlainLopilix, causal_softmax, choose_experts, gated_memory, gelu_erf, read_streams, rotate_halves, rotate_neighbours, silu,
                           unit_rms, write_streams)
from test_gpu_vifelix import _batch, _ops, _run
from tiny_lopilix import (ONE_PASS, ONLY_ATTENTION, ONLY_LATENT, ONLY_MEMORY, TINY_A, TINY_B, attention, dense, latent, layer, make_lopilix_dir, memory,
                          model, moe)

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEV = "cuda:0"


# ----------------------------------------------------------------------------- single kernels
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("S,D", [(1, 64), (2, 20), (2, 4096), (3, 50), (4, 2048), (4, 8000), (5, 128), (7, 30), (16, 1100), (3, 1028)])
def test_stream_norm_kernel(S, D, dtype, tol):
    """A result taken into the streams, the next sublayer's sum read out of them and normed: with and without a gate, without an update,
    without a norm; all rows and only the wanted ones (which leave the streams as they are)."""
    from llmengine_b200.engine.batch import StepBatch
    from llmengine_b200.engine.plan import StreamUpdate
    ops = _ops()
    g = torch.Generator().manual_seed(S * 1000 + D)
    T = 6
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, y, gate = rnd(T, S, D), 3 * rnd(T, D), rnd(T, D).to(dtype)
    mix, put, read, bias, gain = rnd(S, S), rnd(S), rnd(S), rnd(D), 1 + 0.3 * rnd(D)
    dev = lambda t: t.to(DEV)
    new = write_streams(x.double(), mix.double(), put.double(), 1.0, (y * torch.sigmoid(gate.float() + bias)).double())
    ungated = write_streams(x.double(), mix.double(), put.double(), 1.0, y.double())
    want = lambda xs: unit_rms(read_streams(xs, read.double()), 1e-5) * gain.double()
    rows = torch.tensor([5, 0, 3], dtype=torch.int32, device=DEV)
    some = StepBatch.bare(T, torch.device(DEV), logit_rows=rows, logits=torch.zeros(3, 4, device=DEV))
    near = lambda a, b, t=tol: float((a.double().cpu() - b).abs().max()) < t * max(1.0, float(b.abs().max()))
    for update, after in ((StreamUpdate(dev(y), dev(gate), dev(bias), dev(mix), dev(put)), new), (StreamUpdate(dev(y), None, None, dev(mix), dev(put)), ungated),
                          (None, x.double())):
        xd, out = dev(torch.cat([x, x[:1]])).view(T + 1, S * D).clone(), torch.zeros(T + 1, D, dtype=dtype, device=DEV)
        pad = lambda t: None if t is None else torch.cat([t, t[:1]])
        up = None if update is None else StreamUpdate(pad(update.y), pad(update.gate), update.bias, update.mix, update.put)
        _run(ops, lambda p: p.stream_norm(xd, streams=S, read=dev(read), gain=dev(gain), eps=1e-5, out=out, update=up), _batch([T], [0]))
        assert near(out[:T], want(after)) and float(out[T].abs().max()) == 0.0
        assert near(xd[:T].view(T, S, D), after, 1e-5 if dtype == torch.float32 else 1e-4) and torch.equal(xd[T].view(S, D).cpu(), x[0])
        xd, out = dev(x).view(T, S * D).clone(), torch.zeros(T, D, dtype=dtype, device=DEV)
        _run(ops, lambda p: p.stream_norm(xd, streams=S, read=dev(read), gain=dev(gain), eps=1e-5, out=out, update=update, rows="logits"), some)
        assert near(out[:3], want(after)[[5, 0, 3]]) and float(out[3:].abs().max()) == 0.0 and torch.equal(xd.view(T, S, D).cpu(), x)
        if update is not None:
            xd = dev(x).view(T, S * D).clone()
            _run(ops, lambda p: p.stream_norm(xd, streams=S, read=None, gain=None, eps=0.0, out=None, update=update), _batch([T], [0]))
            assert near(xd.view(T, S, D), after, 1e-5 if dtype == torch.float32 else 1e-4)


@pytest.mark.parametrize("H,n,p,room", [(2, 8, 16, 0), (3, 6, 5, 0), (2, 32, 48, 40), (1, 200, 9, 30), (2, 64, 33, 8), (1, 40, 3, 4), (4, 128, 64, 20),
                                        (2, 20, 130, 9), (1, 500, 6, 6)])
def test_recurrence_with_a_forget_gate_per_row(H, n, p, room):
    """S = diag(f) S + (1 - f) v^T, single tokens beside portions down to two tokens and long portions cut into pieces; gates that reach 0
    (the row is replaced) and 1 (the row is kept); the second step starts every request from the state the first one left."""
    ops = _ops()
    g = torch.Generator().manual_seed(n + p)
    lens, cuts, slots = [431, 1, 128, 65, 2, 700], [300, 0, 64, 0, 1, 0], [1, 3, 0, 5, 2, 6]
    scratch = torch.full((room * H * (p * n + n),), float("nan"), device=DEV) if room else None
    mk = lambda *s: torch.randn(*s, generator=g)
    q, v = [mk(L, H * n) for L in lens], [mk(L, H * p) for L in lens]
    f = [1.0 - 0.3 * torch.rand(L, H * n, generator=g) ** 2 for L in lens]
    for r, L in enumerate(lens):
        f[r][L // 3::41, ::3] = 0.0
        f[r][L // 4::7, 1::3] = 1.0
    state = torch.zeros(max(slots) + 2, H, p, n, device=DEV)
    got = [[] for _ in lens]
    for step in range(2):
        spans = [(r, 0, cuts[r]) if step == 0 else (r, cuts[r], lens[r]) for r in range(len(lens))]
        spans = [s for s in spans if s[2] > s[1]]
        cat = lambda xs: torch.cat([xs[r][a:b] for r, a, b in spans]).to(DEV)
        T = sum(b - a for _, a, b in spans)
        out = torch.zeros(T, H * p, device=DEV)
        _run(ops, lambda pl: pl.recurrence(q=cat(q), k=cat(f), v=cat(v), state=state, out=out, heads=H, n=n, p=p, qk_groups=H, scratch=scratch, forget=True),
             _batch([b - a for _, a, b in spans], [slots[r] for r, _, _ in spans]))
        at = 0
        for r, a, b in spans:
            got[r].append(out[at:at + b - a].cpu())
            at += b - a
    for r, L in enumerate(lens):
        want, S = gated_memory(q[r].view(L, H, n).double(), f[r].view(L, H, n).double(), v[r].view(L, H, p).double())
        y = torch.cat(got[r]).view(L, H, p)
        assert float((y - want).abs().max()) < 2e-5 * max(1.0, float(want.abs().max())), r
        assert float((state[slots[r]].cpu() - S.transpose(1, 2)).abs().max()) < 2e-5 * max(1.0, float(S.abs().max())), r
    assert float(state[max(slots) + 1].abs().max()) == 0.0 and float(state[4].abs().max()) == 0.0


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 3e-2)])
def test_small_records_of_the_design(dtype, tol):
    """Embedding with learned positions into several streams; forget gates; a norm per head without a gate."""
    ops = _ops()
    g = torch.Generator().manual_seed(5)
    rnd = lambda *s: torch.randn(*s, generator=g)
    for D, S in ((24, 3), (30, 1), (1040, 2), (300, 5)):
        table, pos, ids, at = rnd(11, D).to(dtype), rnd(9, D).to(dtype), [3, 10, 0, 0, 7, 5], [0, 8, 3, 4, 1, 1]
        b = _batch([6], [0], positions=at)
        b.token_ids.copy_(torch.tensor(ids, dtype=torch.int32))
        out = torch.full((7, S * D), 7.0, device=DEV)
        _run(ops, lambda p: p.embedding(table.to(DEV), out, scale=1.5, positions=pos.to(DEV), streams=S), b)
        want = (table[ids].float() * 1.5 + pos[at].float())[:, None, :].expand(6, S, D).reshape(6, S * D)
        assert float((out[:6].cpu() - want).abs().max()) < 1e-6 and float((out[6] - 7.0).abs().max()) == 0.0
    for T, C in ((3, 20), (5, 33), (200, 512)):
        wide, bias, low = (4 * rnd(T, 2 * C + 3)), rnd(C), torch.rand(C, generator=g)
        wide[0, C] = 90.0
        wide[1, C] = -90.0
        low[-1] = 0.0
        w, q, f = wide.to(DEV), torch.zeros(T, C, device=DEV), torch.zeros(T, C, device=DEV)
        _run(ops, lambda p: p.forget_gates(q_in=w[:, :C], f_in=w[:, C:2 * C], f_bias=bias.to(DEV), lower=low.to(DEV), q=q, f=f), _batch([T], [0]))
        assert float((q.cpu() - silu(wide[:, :C])).abs().max()) < 1e-5
        assert float((f.cpu() - (low + (1 - low) * torch.sigmoid(wide[:, C:2 * C] + bias))).abs().max()) < 1e-6
        assert float(f.max()) <= 1.0 and float((f[1, 0].cpu() - low[0]).abs()) < 1e-6
    for T, groups, group in ((7, 3, 5), (7, 4, 32), (7, 2, 300), (7, 1, 1500), (999, 10, 128), (1201, 9, 20)):
        cols = groups * group
        y, w = 3 * rnd(T, cols), 1 + 0.2 * rnd(cols)
        out = torch.zeros(T + 1, cols, dtype=dtype, device=DEV)
        _run(ops, lambda p: p.gated_norm(y=y.to(DEV), gate=None, weight=w.to(DEV), out=out, group=group, gate_first=False, eps=1e-5), _batch([T], [0]))
        want = unit_rms(y.view(T, groups, group), 1e-5).reshape(T, cols) * w
        assert float((out[:T].float().cpu() - want).abs().max()) < tol * max(1.0, float(want.abs().max())) and float(out[T].abs().max()) == 0.0


@pytest.mark.parametrize("T", [5, 64, 65, 200])
@pytest.mark.parametrize("E,top,groups", [(8, 3, (4, 3)), (6, 2, (3, 1)), (6, 2, (6, 3)), (12, 3, (2, 1)), (9, 9, (3, 3)), (64, 9, (8, 3)), (150, 6, (50, 7)),
                                          (320, 10, (4, 2)), (5, 2, (1, 1))])
def test_routing_by_the_two_best_of_a_group(E, top, groups, T):
    ops = _ops()
    g = torch.Generator().manual_seed(E + T)
    wide = (torch.randn(T, E + 3, generator=g) * 1.5).to(DEV)
    experts, weights = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
    offsets, counts = torch.zeros(E + 1, dtype=torch.int32, device=DEV), torch.zeros(E, dtype=torch.int32, device=DEV)
    order = torch.zeros(T * top, dtype=torch.int32, device=DEV)
    idx, s, margin = choose_experts(wide[:, :E].cpu(), top, groups)
    clear = margin > 1e-4                          # (positions where rounding decides prove nothing)
    assert int(clear.sum()) > 0.8 * T
    for _ in range(2):                             # (the second launch finds the counters as it needs them)
        _run(ops, lambda p: p.moe_route(logits=wide[:, :E], top_k=top, scale=1.7, experts=experts, weights=weights, offsets=offsets, order=order,
                                        counts=counts, mode="sigmoid", groups=groups), _batch([T], [0]))
    assert torch.equal(experts.cpu().long()[clear], idx[clear])
    picked = s.gather(1, idx)
    want = picked / (picked.sum(-1, keepdim=True) + 1e-20) * 1.7
    assert float((weights.cpu() - want)[clear].abs().max()) < 1e-6 and int(counts.abs().max()) == 0
    off, od, ex = offsets.cpu().tolist(), order.cpu().tolist(), experts.cpu().reshape(-1).tolist()
    for e in range(E):
        assert sorted(od[off[e]:off[e + 1]]) == [i for i in range(T * top) if ex[i] == e]


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 4e-2)])
@pytest.mark.parametrize("kernels", ["fast", "tcgen05", "mma"])
@pytest.mark.parametrize("T,E,top,n,k", [(3, 5, 2, 24, 40), (150, 4, 3, 72, 64), (40, 3, 1, 20, 36), (300, 6, 4, 264, 192)])
def test_grouped_products_with_gelu(dtype, tol, T, E, top, n, k, kernels):
    ops = _ops(kernels if kernels == "fast" else {"grouped_linear": kernels})
    g = torch.Generator().manual_seed(T)
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    order = torch.argsort(choice.reshape(-1), stable=True)
    offsets = torch.cat([torch.zeros(1, dtype=torch.long), torch.cumsum(torch.bincount(choice.reshape(-1), minlength=E), 0)])
    x, up, down = (2 * torch.randn(T, k, generator=g)).to(dtype), (torch.randn(E, n, k, generator=g) / math.sqrt(k)).to(dtype), \
        (torch.randn(E, k, n, generator=g) / math.sqrt(n)).to(dtype)
    act, mid = torch.zeros(T * top, n, dtype=dtype, device=DEV), torch.zeros(T * top, n, dtype=dtype, device=DEV)
    y, rows = torch.full((T * top, k), float("nan"), device=DEV), torch.zeros(T * top, k, dtype=dtype, device=DEV)
    lists = dict(offsets=offsets.to(torch.int32).to(DEV), order=order.to(torch.int32).to(DEV), top_k=top)

    def records(p):
        p.grouped_linear(x=x.to(DEV), w=up.to(DEV), out=act, gather=True, scatter=False, mid=mid, act="gelu", rows=rows, **lists)
        p.grouped_linear(x=act, w=down.to(DEV), out=y, gather=False, scatter=True, **lists)
    _run(ops, records, _batch([T], [0]))
    if "moe_tcgen05" in ops._libs:
        assert ops.grouped_tcgen05_status() == 0
    for i, e in enumerate(choice.reshape(-1).tolist()):
        a = gelu_erf(up[e].float() @ x[i // top].float()).to(dtype).float()
        assert float((y[i].cpu() - down[e].float() @ a).abs().max()) < tol * 3, (i, e)


def _maps_case(ops, dtype, G, rep, dk, dv, page, lens, cuts, rot, interleaved=True, seed=0):
    """Differential attention (2 G key heads in pairs on G value heads, `rep` query heads each, norm per head before the rotation, the
    difference of the maps and its norm): requests of `lens` tokens whose first `cuts[r]` tokens are cached by one step; the second step brings the rest.
    Returns (the engine's output of the second step, the plain result for those tokens)."""
    from llmengine_b200.engine.batch import GroupView, StepBatch
    from llmengine_b200.parts.latent import PartialRotaryEncoding
    g = torch.Generator().manual_seed(seed)
    R, ps, H, K = len(lens), page, 2 * G * rep, 2 * G
    eps, scale = 1e-5, 1.7 / math.sqrt(dk)
    q_gain, k_gain = 1 + 0.2 * torch.randn(dk, generator=g), 1 + 0.2 * torch.randn(dk, generator=g)
    proj = [(torch.randn(n, H * dk + K * dk + G * dv, generator=g) * 1.5).to(dtype) for n in lens]
    blocks = [-(-n // ps) for n in lens]
    perm = torch.randperm(sum(blocks) + 3, generator=g).tolist()
    tables = torch.full((R, max(blocks) + 1), -1, dtype=torch.int32)
    at = 0
    for r, nb in enumerate(blocks):
        tables[r, :nb] = torch.tensor(perm[at:at + nb], dtype=torch.int32)
        at += nb
    cache = torch.full((sum(blocks) + 3, ps * (K * dk + G * dv)), float("nan"), dtype=dtype, device=DEV)
    f = PartialRotaryEncoding.build_frequencies(rot, 500.0) if rot else None
    qs, ks = H * dk, K * dk
    for step in range(2):
        spans = [(0, cuts[r]) if step == 0 else (cuts[r], lens[r]) for r in range(R)]
        spans = [(r, a, b) for r, (a, b) in enumerate(spans) if b > a]
        rows = torch.cat([proj[r][a:b] for r, a, b in spans]).to(DEV)
        T = rows.shape[0]
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        slots = [int(tables[r, p // ps]) * ps + p % ps for r, a, b in spans for p in range(a, b)]
        q_lens = [b - a for _, a, b in spans]
        batch = StepBatch(
            num_tokens=T, num_requests=len(spans), q_lens=q_lens, start_positions=[a for _, a, _ in spans], token_ids=i32([0] * T),
            positions=i32([p for _, a, b in spans for p in range(a, b)]), token_request=i32([r for r, a, b in spans for _ in range(a, b)]),
            cu_q_lens=i32([0] + list(np.cumsum(q_lens))), ctx_lens=i32([b for _, _, b in spans]),
            state_slots=i32([r for r, _, _ in spans]), first_portion=i32([int(a == 0) for _, a, _ in spans]), logit_rows=i32([]),
            decode_rows=i32([i for i, q in enumerate(q_lens) if q == 1]), portion_rows=i32([i for i, q in enumerate(q_lens) if q != 1]),
            groups=[GroupView(ps, 0, tables.to(DEV), i32(slots), tables.shape[1])])
        q, out = torch.zeros(T, H * dk, dtype=dtype, device=DEV), torch.zeros(T, H * dv, dtype=dtype, device=DEV)
        heads = torch.full((T, G * rep * dv), float("nan"), dtype=dtype, device=DEV)
        room = torch.full((max(512, R * G * ((rep + 7) // 8)) * 16 * (dv + 2),), float("nan"), device=DEV)
        _run(ops, lambda p: p.window_attention(
            q_in=rows[:, :qs], k_in=rows[:, qs:qs + ks], v_in=rows[:, qs + ks:], q_gain=q_gain.to(DEV), k_gain=k_gain.to(DEV), eps=eps,
            inv_freq=f.to(DEV) if rot else None, rot_dims=rot or 0, amplitude=1.0, q=q, out=out, cache=cache, group=0, num_heads=H, num_kv_heads=K,
            qk_dim=dk, v_dim=dv, window=0, keep_first=0, scale=scale, head_norm=True, value_share=2, interleaved=interleaved,
            scratch=torch.zeros(R * H * 8 * (dv + 2), device=DEV) if dtype == torch.bfloat16 else None, difference=(0.6, 0.4, 1e-5), heads=heads,
            maps_scratch=room if dtype == torch.bfloat16 else None), batch)
    want, rt = [], lambda t: t.to(dtype).float()
    turn = rotate_neighbours if interleaved else rotate_halves
    for r, a, b in spans:
        n, pr = lens[r], proj[r].float()
        fin = lambda x, heads, gain: rt(turn(unit_rms(x.view(n, heads, dk), eps) * gain, torch.arange(n), {"dims": rot, "base": 500.0}) if rot
                                        else unit_rms(x.view(n, heads, dk), eps) * gain)
        qq, kk, vv = fin(pr[:, :qs], H, q_gain), fin(pr[:, qs:qs + ks], K, k_gain), pr[:, qs + ks:].view(n, G, dv)
        p = causal_softmax(torch.einsum("ihd,jhd->hij", qq, kk.repeat_interleave(rep, 1)) * scale)
        m = torch.einsum("hij,jhd->ihd", p, vv.repeat_interleave(2 * rep, 1)).view(n, G, 2, rep, dv)
        want.append((unit_rms(m[:, :, 0] - 0.6 * m[:, :, 1], 1e-5) * 0.4).reshape(n, G * rep * dv)[a:b])
    return heads.float().cpu(), torch.cat(want)


@pytest.mark.parametrize("kernels", ["fast", "plain"])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("G,rep,dk,dv,page,rot,interleaved", [
    (2, 2, 32, 64, 16, 16, True), (1, 4, 64, 128, 64, 32, True), (2, 1, 64, 128, 16, 64, True), (1, 3, 10, 6, 8, 6, True), (3, 1, 48, 96, 32, 20, True),
    (2, 3, 16, 48, 64, None, True), (1, 2, 64, 64, 16, 16, False), (1, 1, 128, 128, 16, 64, True), (2, 4, 64, 128, 128, 8, False), (1, 16, 64, 128, 8, 32, True), (2, 3, 64, 128, 16, 32, True), (1, 9, 32, 32, 24, 8, True)])
def test_differential_attention_kernels(kernels, dtype, tol, G, rep, dk, dv, page, rot, interleaved):
    """Portions that start inside a page, single tokens beside them whose keys are cut into ranges, requests of one token; free pages hold
    NaN, and so does every place of a held page that no token has been written to."""
    ops = _ops(kernels)
    lens, cuts = [700, 9, 1, 650, 131, 77, 300], [699, 0, 0, 640, 130, 70, 3]
    got, want = _maps_case(ops, dtype, G, rep, dk, dv, page, lens, cuts, rot, interleaved, seed=dk + dv)
    assert torch.isfinite(got).all()
    assert float((got - want).abs().max()) < tol
    if kernels == "fast" and dtype == torch.bfloat16:
        assert (f"attention_maps@DK={dk},DV={dv}" in ops._libs) == (dk % 16 == 0 and dv % 16 == 0)
        tc = "attention_tc@HEAD_DIM=64,VALUE_DIM=128,MAPS=2"
        assert (tc in ops._libs) == ((dk, dv) == (64, 128))
        if tc in ops._libs:
            assert ops._libs[tc].llme_attention_tc_status() == 0, "no bounded wait gave up"


# ----------------------------------------------------------------------------- each mixer in a model of its own
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg", [("memory", ONLY_MEMORY), ("attention", ONLY_ATTENTION), ("latent", ONLY_LATENT), ("one pass", ONE_PASS)])
def test_each_mixer_alone(tmp_path, name, cfg, dtype):
    d = make_lopilix_dir(str(tmp_path / "m"), cfg, seed=9)
    replay_all_schedules(d, cfg, dtype, [70, 5, 120, 1, 2], 16, None, DEV, only=("whole", "bulk_then_single", "portions"))


# ----------------------------------------------------------------------------- every schedule
# sizes the tensor-core kernels take: maps of 64 on values of 128 and of 32, latents of 64 and 192, memories of 64 and 128 rows
BIG = model(131, 128, 4, 400, 1e-6, 0.7, 1.4, [
    layer("attention", attention(4, 2, 64, 128, 0.125, 0.45, base=5000.0, dims=32), moe(6, 2, 64, 1.3, groups=(2, 1))),
    layer("hgrn2", memory(3, 64, 32), dense(192)),
    layer("latent_attention", latent(5, 32, 16, 48, 192, 0.15, base=900.0, scaling=(4.0, 64, 8.0, 1.0)), moe(8, 3, 72, 2.0)),
    layer("hgrn2", memory(2, 128, 64), dense(96)),
    layer("attention", attention(6, 2, 32, 32, 0.2, 0.8, base=300.0, dims=20)),
    layer("latent_attention", latent(2, 16, 32, 32, 64, 0.2, base=100.0), dense(160)),
], loop=(1, 3, 2))


@pytest.mark.parametrize("kernels", ["fast", "plain"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,cfg,page,lens", [
    ("A", TINY_A, 16, [70, 33, 50, 1, 19, 64]),
    ("B", TINY_B, 8, [2, 5, 64, 90, 48]),
    ("M", ONLY_MEMORY, 64, [150, 3, 40, 64, 7]),
    ("BIG", BIG, 64, [150, 40, 129, 2, 64]),
    ("BIG16", BIG, 16, [150, 40, 129, 2, 64]),
])
def test_replay_gpu(tmp_path, name, cfg, page, lens, dtype, kernels):
    d = make_lopilix_dir(str(tmp_path / name), cfg, seed=11)
    worst = replay_all_schedules(d, cfg, dtype, lens, page, None, DEV, kernels=kernels)
    print(f"replay {name} {dtype} {kernels}: share of the tolerance: " + ", ".join(f"{k} {v:.2f}" for k, v in worst.items()))


# ----------------------------------------------------------------------------- constants that are one off
EDGE = model(50, 64, 2, 128, 1e-5, 0.8, 1.5, [
    layer("attention", attention(4, 2, 32, 64, 0.2, 0.4, base=200.0, dims=8), moe(8, 3, 32, 1.5, groups=(4, 2))),
    layer("latent_attention", latent(3, 16, 16, 16, 64, 0.3, base=60.0, scaling=(4.0, 32, 4.0, 1.0)), dense(40)),
    layer("hgrn2", memory(2, 16, 16), dense(48)),
], loop=(0, 2, 2))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_constants_that_are_one_off(tmp_path, dtype):
    """Other rotated coordinates, another base, scale, stretching or difference, one expert fewer, other groups, another multiplier of
    the results, another number of passes, a loop over other layers: each moves the plain implementation's logits far beyond the
    tolerance.  The engine, with the right constants, stays within it at every position, in prompts and decoded."""
    d = make_lopilix_dir(str(tmp_path / "edge"), EDGE, seed=31)
    reqs = {"a": random_ids(90, 50, 1), "b": random_ids(23, 50, 2), "c": random_ids(5, 50, 3)}
    ref, tol = reference_logits(d, reqs, dtype)
    router = lambda c: c["layers"][0]["mlp"]["router"]
    mixer = lambda c, i: c["layers"][i]["mixer"]
    changes = {
        "more coordinates rotated": lambda c: mixer(c, 0)["rot"].__setitem__("dims", 16),
        "another base": lambda c: mixer(c, 0)["rot"].__setitem__("base", 4.0),
        "another scale": lambda c: mixer(c, 0).__setitem__("scale", 0.8),
        "another difference": lambda c: mixer(c, 0).__setitem__("diff", 0.8),
        "not stretched": lambda c: mixer(c, 1)["rot"].pop("scaling"),
        "stretched more": lambda c: mixer(c, 1)["rot"]["scaling"].__setitem__("factor", 16.0),
        "a latent scale": lambda c: mixer(c, 1).__setitem__("scale", 1.0),
        "one expert per token": lambda c: router(c).__setitem__("top", 1),
        "one group kept": lambda c: router(c).__setitem__("groups", {"count": 2, "keep": 1}),
        "no groups": lambda c: router(c).pop("groups"),
        "another router scale": lambda c: router(c).__setitem__("scale", 0.5),
        "another multiplier": lambda c: c.__setitem__("residual_mult", 1.1),
        "logits not scaled": lambda c: c.__setitem__("logit_scale", 1.0),
        "one more pass": lambda c: c["loop"].__setitem__("times", 3),
        "no loop": lambda c: c.pop("loop"),
        "a loop over one layer": lambda c: c["loop"].__setitem__("start", 1),
        "another eps": lambda c: c["norm"].__setitem__("eps", 0.5),
    }
    for what, change in changes.items():
        other = PlainLopilix(variant_dir(d, str(tmp_path / what.replace(" ", "_")), change))
        moved = float((other.logits(reqs["a"]) - ref["a"]).abs().max())
        assert moved > 3 * tol, f"{what} moves the logits by {moved:.3g} only (tolerance {tol:.3g})"
    for page in (4, 16, 64):
        for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_bulk_then_single(reqs, 60)), ("portions", trace_portions(reqs))):
            eng = engine_for(d, dtype, 256, page_size=page, max_requests=2, max_model_len=128)
            compare(replay(eng, steps, poison=True), ref, tol, f"{dtype}/page {page}/{what}")


def _far_token_inputs(w, token, read):
    """Edits embedding and norm so that every input has a part (coordinate 0) that does not depend on the token, and returns a
    direction that is large on `token` alone among the tokens' normed inputs of layer 0."""
    e = w["embed"].float()
    e[:, 0] = 0.8
    pos = w["pos"].float() * 0.02
    pos[:, 0] = 0.0
    gain = w["l0.norm1"].float()
    gain[0] = 1.0
    w.update({"embed": e.to(torch.bfloat16), "pos": pos.to(torch.bfloat16), "l0.norm1": gain.to(torch.bfloat16), "l0.hc1.in": torch.tensor(read).to(torch.bfloat16)})
    h = unit_rms(w["embed"].float() * float(sum(read)), 1e-5) * gain
    probe = torch.linalg.lstsq(h, torch.nn.functional.one_hot(torch.tensor(token), h.shape[0]).float()[:, None]).solution[:, 0]
    return probe / (probe @ h[token])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,dk", [("maps", 16), ("maps", 64), ("latent", 24), ("latent", 64)])
def test_a_key_far_back_among_hundreds(tmp_path, dtype, kind, dk):
    """One token's key points along a coordinate that is not rotated (in the first map alone, in a latent coordinate of its own), and every
    query points there too.  Put at position 3 of 400 it still takes most of the attention at the end, over page borders: exchanging
    it moves the last logits by many tolerances, in the plain implementation and, within the tolerance of it, in the engine."""
    read = [0.7, 0.5]
    if kind == "maps":
        H, G = 4, 2
        mixer = attention(H, G, dk, 2 * dk, 14.0 / dk, 0.4, base=100.0, dims=8)
    else:
        H = 3
        mixer = latent(H, dk, 8, 16, dk, 0.4, base=100.0)
    cfg = model(40, 48, 2, 512, 1e-5, 1.0, 1.0, [layer("attention" if kind == "maps" else "latent_attention", mixer, dense(24))])

    def change(w):
        probe = _far_token_inputs(w, 7, read)
        q = w["l0.mix.q"].float() * 0.3
        if kind == "maps":
            k = w["l0.mix.k"].float() * 0.5
            for b in range(G):
                k[2 * b * dk + dk - 1] = 6.0 * probe          # the first map's last coordinate
            for a in range(H):
                q[2 * a * dk + dk - 1] = 0.0
                q[2 * a * dk + dk - 1, 0] = 6.0
            w["l0.mix.k"] = k.to(torch.bfloat16)
        else:
            low, uk = w["l0.mix.dkv"].float() * 0.5, w["l0.mix.uk"].float() * 0.3
            low[0] = 6.0 * probe                              # the latent's first coordinate
            for a in range(H):
                uk[(a + 1) * dk - 1] = 0.0
                uk[(a + 1) * dk - 1, 0] = 4.0
                at = a * (dk + 8) + dk - 1
                q[at] = 0.0
                q[at, 0] = 2.5
            w.update({"l0.mix.dkv": low.to(torch.bfloat16), "l0.mix.uk": uk.to(torch.bfloat16)})
        w["l0.mix.q"] = q.to(torch.bfloat16)
    d_ = make_lopilix_dir(str(tmp_path / "m"), cfg, seed=3, change=change)
    ids = [t if t != 7 else 8 for t in random_ids(400, 40, 5)]
    ids[3] = 7
    reqs = {"a": ids, "b": ids[:70]}
    ref, tol = reference_logits(d_, reqs, dtype)
    without = list(ids)
    without[3] = 9
    plain = PlainLopilix(d_)
    moved = float((plain.logits(ids)[-1] - plain.logits(without)[-1]).abs().max())
    assert moved > 10 * tol, f"the far token moves the logits by {moved:.3g} (tolerance {tol:.3g})"
    for page in (16, 64):
        for what, steps in (("whole", trace_whole(reqs)), ("decoded", trace_bulk_then_single(reqs, 40)), ("portions", trace_portions(reqs))):
            eng = engine_for(d_, dtype, 512, page_size=page, max_requests=2, max_model_len=512)
            compare(replay(eng, steps, poison=True), ref, tol, f"{dtype}/page {page}/{what}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_first_token_that_only_the_memory_remembers(tmp_path, dtype):
    """Memories alone, gates near one, in a loop whose every pass has a state of its own: changing the FIRST token of a prompt of 200 still
    moves the last logits, so a state that is lost, zeroed, shared between passes or taken from another slot on the way (portions,
    single tokens, slots used again) would show there."""
    cfg = model(45, 48, 2, 400, 1e-5, 0.9, 1.2, [layer("hgrn2", memory(4, 32, 16), dense(40)), layer("hgrn2", memory(3, 40, 16))], loop=(0, 1, 2))

    def change(w):
        for i in (0, 1):
            w[f"l{i}.mix.lower"] = torch.full_like(w[f"l{i}.mix.lower"], 0.97)
            w[f"l{i}.mix.f.b"] = torch.full_like(w[f"l{i}.mix.f.b"], 1.5)
    d = make_lopilix_dir(str(tmp_path / "m"), cfg, seed=6, change=change)
    reqs = {f"r{i}": random_ids(n, 45, 70 + i) for i, n in enumerate([200, 40, 170, 9, 130])}
    ref, tol = reference_logits(d, reqs, dtype)
    other = list(reqs["r0"])
    other[0] = (other[0] + 1) % 45
    if dtype == "float32":      # bfloat16 rounding of hundreds of tokens' writes moves these logits more than the first token does
        assert float((PlainLopilix(d).logits(other)[-1] - ref["r0"][-1]).abs().max()) > 5 * tol
    for what, steps in schedules(reqs, tail=40).items():
        eng = engine_for(d, dtype, max_live_tokens(steps, 64), page_size=16, max_requests=4, max_model_len=400)
        compare(replay(eng, steps, poison=True), ref, tol, f"far/{dtype}/{what}")


# ----------------------------------------------------------------------------- from the first token on, for long
@pytest.mark.parametrize("cfg_name", ["A", "M"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoding_from_the_first_token_through_captured_steps(tmp_path, dtype, cfg_name):
    """Three requests decoded token by token from position 0 on, over several pages, with the steps captured in CUDA graphs: the same
    logits as whole prompts.  Also for a model that keeps no pages at all."""
    from llmengine_b200.engine.engine import StepEntry
    cfg = TINY_A if cfg_name == "A" else ONLY_MEMORY
    d = make_lopilix_dir(str(tmp_path / "m"), cfg, seed=13)
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
    d = make_lopilix_dir(str(tmp_path / "m"), TINY_A, seed=5)
    llm = LLM(d, dtype="float32", page_size=16, max_cached_tokens=512, max_num_seqs=4, max_num_batched_tokens=64,
              prefill_chunk=40, max_model_len=256)
    prompts = [random_ids(n, TINY_A["vocab"], i) for i, n in enumerate([1, 5, 64, 90, 33, 7])]
    outs = llm.generate(prompts, SamplingParams(greedy=True), max_tokens=12, eos_token_id=None)
    plain = PlainLopilix(d)
    for p, o in zip(prompts, outs):
        assert o.token_ids == greedy_by_the_plain_model(plain, p, 12)
    llm.engine.cache.check_invariants()
    assert not llm.engine.cache.requests and llm.scheduler.all_done()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_program(tmp_path, dtype):
    cfg = TINY_A
    d = make_lopilix_dir(str(tmp_path / "m"), cfg, seed=17)
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
