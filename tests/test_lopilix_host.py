"""The Lopilix design on the host: configuration, the order of a loop, tensor names, the cache a layer asks for, the plain
implementation's mechanisms on inputs whose result can be written down, and the engine's own logic (batch metadata, pages,
state slots, scheduling) with a CPU stand-in for the kernels, against the plain implementation."""
import copy
import math

import pytest
import torch

from helpers import random_ids
from host_ops import HostOps
from llmengine_b200 import LLM, SamplingParams
from llmengine_b200.config import ConfigError, LopilixConfig, config_from_dict
from llmengine_b200.engine.model import Model
from llmengine_b200.parts import Runtime
from llmengine_b200.parts.base import StatesSpec
from llmengine_b200.parts.latent import PartialRotaryEncoding
from lopilix_cases import greedy_by_the_plain_model, replay_all_schedules
from plain_lopilix import (PlainLopilix, causal_softmax, choose_experts, dense_ff, difference_attention, difference_weight, frequencies,
                           gated, gated_memory, gelu_erf, latent_attention, memory_mixer, read_streams, rotate_halves, rotate_neighbours,
                           routed_ff, runs, silu, unit_rms, write_streams)
from tiny_lopilix import ONE_PASS, ONLY_ATTENTION, ONLY_LATENT, ONLY_MEMORY, TINY_A, TINY_B, make_lopilix_dir, tensor_shapes

ALL = [("A", TINY_A), ("B", TINY_B), ("M", ONLY_MEMORY), ("T", ONLY_ATTENTION), ("L", ONLY_LATENT), ("P", ONE_PASS)]


def test_every_size_and_constant_comes_from_the_file():
    c = config_from_dict(TINY_A)
    assert isinstance(c, LopilixConfig) and (c.hidden_size, c.vocab_size, c.streams, c.max_positions, c.norm_eps) == (64, 101, 3, 600, 1e-5)
    assert (c.residual_mult, c.logit_scale) == (0.8, 1.7)
    m, a, l = c.mixers[:3]
    assert (m.heads, m.dim, m.vdim) == (3, 24, 40)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.diff, a.rot.base, a.rot.dims, a.rot.scaling) == (4, 2, 32, 64, 0.2, 0.35, 500.0, 16, None)
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.scale, l.rot.base, l.rot.dims) == (3, 16, 8, 24, 64, 0.25, 300.0, 8)
    assert (l.rot.scaling.factor, l.rot.scaling.original, l.rot.scaling.fast, l.rot.scaling.slow) == (8.0, 64, 8.0, 1.0)
    f = c.mlps
    assert (f[1].kind, f[1].ff) == ("dense", 96)
    assert (f[0].ff, f[0].experts, f[0].top, f[0].scale, f[0].groups, f[0].keep) == (40, 9, 2, 1.5, 3, 2)
    b = config_from_dict(TINY_B)
    assert (b.mlps[1].groups, b.mlps[1].keep) == (1, 1) and b.mlps[2] is None
    for _, cfg in ALL:
        assert config_from_dict(config_from_dict(cfg).to_dict()) == config_from_dict(cfg)
    for path in (["width"], ["streams"], ["max_positions"], ["norm", "eps"], ["residual_mult"], ["logit_scale"], ["layers", 0, "mixer", "vdim"],
                 ["layers", 1, "mixer", "diff"], ["layers", 1, "mixer", "scale"], ["layers", 1, "mixer", "kv_heads"], ["layers", 1, "mixer", "rot", "base"],
                 ["layers", 1, "mixer", "rot", "dims"], ["layers", 2, "mixer", "kv_rank"], ["layers", 2, "mixer", "rot_dim"],
                 ["layers", 2, "mixer", "rot", "scaling", "fast"], ["layers", 0, "mlp", "router", "top"], ["layers", 0, "mlp", "router", "scale"],
                 ["layers", 0, "mlp", "expert"], ["layers", 0, "mlp", "router", "groups", "keep"], ["layers", 1, "mlp", "ff"], ["layers", 2, "type"],
                 ["loop", "times"]):
        e = copy.deepcopy(TINY_A)
        at = e
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=str(path[-1])):
            config_from_dict(e)
    for edit, word in ((lambda e: e["layers"][1]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
                       (lambda e: e["layers"][1]["mixer"]["rot"].__setitem__("dims", 34), "rot.dims"),
                       (lambda e: e["layers"][2]["mixer"]["rot"].__setitem__("dims", 7), "rot.dims"),
                       (lambda e: e["layers"][0]["mlp"]["router"].__setitem__("top", 7), "top"),
                       (lambda e: e["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 4), "count"),
                       (lambda e: e["layers"][0]["mlp"]["router"]["groups"].__setitem__("keep", 4), "keep"),
                       (lambda e: e["loop"].__setitem__("stop", 5), "loop.stop"),
                       (lambda e: e.__setitem__("streams", 0), "streams"),
                       (lambda e: e["layers"][0].__setitem__("type", "something_else"), "something_else"),
                       (lambda e: e["layers"][1]["mlp"].__setitem__("kind", "sparse"), "sparse")):
        e = copy.deepcopy(TINY_A)
        edit(e)
        with pytest.raises(ConfigError, match=word):
            config_from_dict(e)


def test_the_order_of_a_loop():
    """Every pass over the looped layers is a run of its own, with a cache or state of its own; nothing is added between passes."""
    order = lambda cfg: [r.layer for r in config_from_dict(cfg).model_spec().order]
    assert order(TINY_A) == [0, 1, 0, 1, 2, 3] and order(TINY_B) == [0, 1, 1, 1, 2, 3]
    assert order(ONLY_MEMORY) == [0, 1, 1] and order(ONLY_ATTENTION) == [0, 0, 0] and order(ONE_PASS) == [0, 1]
    assert order({k: v for k, v in TINY_A.items() if k != "loop"}) == [0, 1, 2, 3]
    assert order(dict(TINY_A, loop={"start": 2, "stop": 2, "times": 3})) == [0, 1, 2, 3]
    for _, cfg in ALL:
        assert order(cfg) == runs(cfg)
        assert not any(r.add_embedding or r.cache_from is not None for r in config_from_dict(cfg).model_spec().order)


@pytest.mark.parametrize("name,cfg", ALL)
def test_the_model_declares_the_design_s_tensors(name, cfg):
    m = Model(config_from_dict(cfg).model_spec(), Runtime(None, torch.device("cpu"), torch.float32, 1))
    assert {n: tuple(s.shape) for n, s in m.weight_specs().items()} == tensor_shapes(cfg)
    assert m.tied_tensors() == {"head": "embed"}


def test_what_each_layer_keeps_between_steps():
    m = Model(config_from_dict(TINY_A).model_spec(), Runtime(None, torch.device("cpu"), torch.float32, 1))
    specs = [b.cache_spec() for b in m.blocks]
    assert isinstance(specs[0], StatesSpec) and dict(specs[0].parts) == {"state": (3, 40, 24)}
    assert specs[1].paged and (specs[1].num_kv_heads, specs[1].k_dim, specs[1].v_dim, specs[1].value_share) == (4, 32, 64, 2)
    assert specs[1].bytes_per_token(torch.float32) == 4 * (4 * 32 + 2 * 64), "two maps' keys, one set of values"
    assert tuple(specs[1].allocate(3, 16, torch.float32, torch.device("cpu")).shape) == (3, 16 * (4 * 32 + 2 * 64))
    assert specs[2].paged and specs[2].width == 64 + 8, "only the latent and the shared rotated key part"
    assert len(m.cache_specs()) == 6, "every pass of the loop keeps a cache of its own"


# ----------------------------------------------------------------------------- the plain implementation against itself
def test_plain_mechanisms_by_hand():
    assert torch.allclose(unit_rms(torch.tensor([[3.0, 4.0]]), 0.0), torch.tensor([[3.0, 4.0]]) / (12.5 ** 0.5))
    assert abs(float(silu(torch.tensor(1.0))) - 0.7310586) < 1e-6
    assert abs(float(gelu_erf(torch.tensor(1.0))) - 0.8413447) < 1e-6 and abs(float(gelu_erf(torch.tensor(-2.0))) + 0.0455003) < 1e-6
    p = causal_softmax(torch.tensor([[0.0, 9.0, 9.0], [0.0, math.log(3.0), 9.0], [0.0, 0.0, 0.0]]))
    assert torch.allclose(p, torch.tensor([[1.0, 0.0, 0.0], [0.25, 0.75, 0.0], [1 / 3, 1 / 3, 1 / 3]]))
    # rotation: position 0 changes nothing; coordinates from `dims` on pass; the two layouts pair different coordinates
    v = torch.arange(12.0).view(1, 2, 6)
    rot = {"base": 100.0, "dims": 4}
    for turn in (rotate_halves, rotate_neighbours):
        assert torch.equal(turn(v, torch.tensor([0]), rot), v)
        assert torch.equal(turn(v.expand(3, 2, 6), torch.tensor([0, 1, 7]), rot)[..., 4:], v.expand(3, 2, 6)[..., 4:])
    c0, s0, c1, s1 = math.cos(7.0), math.sin(7.0), math.cos(0.7), math.sin(0.7)
    h, n = rotate_halves(v, torch.tensor([7]), rot)[0, 0], rotate_neighbours(v, torch.tensor([7]), rot)[0, 0]
    assert torch.allclose(h[:4], torch.tensor([0 * c0 - 2 * s0, 1 * c1 - 3 * s1, 2 * c0 + 0 * s0, 3 * c1 + 1 * s1]), atol=1e-5)
    assert torch.allclose(n[:4], torch.tensor([0 * c0 - 1 * s0, 1 * c0 + 0 * s0, 2 * c1 - 3 * s1, 3 * c1 + 2 * s1]), atol=1e-5)


def test_stretched_frequencies():
    """Pairs that turn often keep their frequency, pairs that hardly turn get it divided, a ramp between; the amplitude grows with the
    factor's logarithm; the engine's frequencies are the plain ones."""
    sc = {"factor": 4.0, "original": 256, "fast": 8.0, "slow": 1.0}
    f, amp = frequencies(16, 1000.0, sc)
    plain, one = frequencies(16, 1000.0)
    assert one == 1.0 and abs(amp - (0.1 * math.log(4.0) + 1.0)) < 1e-12
    place = lambda t: 16 * math.log(256 / (2 * math.pi * t)) / (2 * math.log(1000.0))
    lo, hi = math.floor(place(8.0)), math.ceil(place(1.0))
    assert 0 < lo < hi < 8
    for i in range(8):
        r = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        assert abs(f[i] - plain[i] * (r / 4.0 + 1.0 - r)) < 1e-9
    assert f[0] == plain[0] and abs(f[7] - plain[7] / 4.0) < 1e-12
    for dims, base, s in ((16, 1000.0, sc), (6, 50.0, None), (32, 500000.0, {"factor": 2.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
                          (8, 30.0, {"factor": 3.0, "original": 4, "fast": 32.0, "slow": 16.0})):
        got = PartialRotaryEncoding.build_frequencies(dims, base, None if s is None else tuple(s[k] for k in ("factor", "original", "fast", "slow")))
        assert torch.allclose(got, torch.tensor(frequencies(dims, base, s)[0]), rtol=1e-5)


def test_the_memory_is_a_sum_over_earlier_tokens():
    """Row c of the state is sum_j (product of f_c over the tokens behind j) (1 - f_c(j)) v_j; a gate of one keeps everything and takes
    nothing, a gate of zero replaces the row by v; handing the state on at a cut changes nothing."""
    g = torch.Generator().manual_seed(0)
    T, d, P = 6, 4, 3
    q, v = torch.randn(T, 1, d, generator=g, dtype=torch.float64), torch.randn(T, 1, P, generator=g, dtype=torch.float64)
    f = torch.rand(T, 1, d, generator=g, dtype=torch.float64)
    f[2, 0, 1], f[3, 0, 1], f[4, 0, 2] = 0.0, 1.0, 0.0
    o, S = gated_memory(q, f, v)
    for t in range(T):
        M = torch.zeros(d, P, dtype=torch.float64)
        for j in range(t + 1):
            M += (f[j + 1:t + 1, 0].prod(0) * (1.0 - f[j, 0]))[:, None] * v[j, 0][None, :]
        assert torch.allclose(o[t, 0], M.t() @ q[t, 0], atol=1e-12)
    first, S1 = gated_memory(q[:2], f[:2], v[:2])
    second, S2 = gated_memory(q[2:], f[2:], v[2:], S1)
    assert torch.allclose(torch.cat([first, second]), o) and torch.allclose(S2, S)
    # the mixer around it, every projection a selection of the input's coordinates
    H, d, P = 2, 3, 2
    D = 2 * H * d + H * P
    eye, h = torch.eye(D, dtype=torch.float64), torch.randn(T, D, generator=g, dtype=torch.float64)
    w = {"p.q": eye[:H * d], "p.f": eye[H * d:2 * H * d], "p.v": eye[2 * H * d:], "p.f.b": torch.randn(H * d, generator=g, dtype=torch.float64),
         "p.lower": torch.rand(H * d, generator=g, dtype=torch.float64), "p.norm": torch.tensor([1.5, 0.5], dtype=torch.float64)}
    got = memory_mixer(h, w, "p.", {"heads": H, "dim": d, "vdim": P}, 1e-5)
    for a in range(H):
        M = torch.zeros(d, P, dtype=torch.float64)
        for t in range(T):
            at = slice(a * d, (a + 1) * d)
            low = w["p.lower"][at]
            fg = low + (1.0 - low) / (1.0 + torch.exp(-(h[t, H * d:2 * H * d][at] + w["p.f.b"][at])))
            M = fg[:, None] * M + (1.0 - fg)[:, None] * h[t, 2 * H * d + a * P:2 * H * d + (a + 1) * P][None, :]
            z = h[t, at]
            o = M.t() @ (z / (1.0 + torch.exp(-z)))
            assert torch.allclose(got[t, a * P:(a + 1) * P], o / torch.sqrt((o * o).mean() + 1e-5) * w["p.norm"], atol=1e-10)


def test_difference_attention_written_out():
    """Two query heads on one key/value head, each with two maps; lambda from its four vectors; the norm without a weight."""
    g = torch.Generator().manual_seed(2)
    T, H, d, P, D = 5, 2, 4, 3, 6
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    w = {"p.q": rnd(H * 2 * d, D), "p.k": rnd(2 * d, D), "p.v": rnd(P, D), "p.q.norm": rnd(d), "p.k.norm": rnd(d),
         **{"p." + n: 0.5 * rnd(d) for n in ("lq1", "lk1", "lq2", "lk2")}}
    h, m = rnd(T, D), {"heads": H, "kv_heads": 1, "dim": d, "vdim": P, "scale": 0.7, "diff": 0.3, "rot": {"base": 20.0, "dims": 2}}
    got = difference_attention(h, w, "p.", m, 1e-4, torch.arange(T), None)
    lam = math.exp(float(w["p.lq1"] @ w["p.lk1"])) - math.exp(float(w["p.lq2"] @ w["p.lk2"])) + 0.3
    assert abs(float(difference_weight(w, "p.", 0.3)) - lam) < 1e-12

    def finished(x, gain, p):
        x = x / torch.sqrt((x * x).mean() + 1e-4) * gain
        u, v = float(x[0]), float(x[1])
        return torch.cat([torch.tensor([u * math.cos(p) - v * math.sin(p), v * math.cos(p) + u * math.sin(p)], dtype=torch.float64), x[2:]])
    vals = [w["p.v"] @ h[j] for j in range(T)]
    for i in range(T):
        for a in range(H):
            maps = []
            for c in (0, 1):
                q = finished(w["p.q"][(2 * a + c) * d:(2 * a + c + 1) * d] @ h[i], w["p.q.norm"], i)
                e = torch.stack([torch.exp(0.7 * (q @ finished(w["p.k"][c * d:(c + 1) * d] @ h[j], w["p.k.norm"], j))) for j in range(i + 1)])
                maps.append(sum(e[j] * vals[j] for j in range(i + 1)) / e.sum())
            o = maps[0] - lam * maps[1]
            assert torch.allclose(got[i, a * P:(a + 1) * P], o / torch.sqrt((o * o).mean() + 1e-4) * 0.7, atol=1e-6)


def test_latent_attention_written_out():
    g = torch.Generator().manual_seed(3)
    T, H, d, dr, P, R, D = 5, 2, 3, 4, 2, 5, 6
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    w = {"p.q": rnd(H * (d + dr), D), "p.dkv": rnd(R + dr, D), "p.dkv.norm": rnd(R), "p.uk": rnd(H * d, R), "p.uv": rnd(H * P, R), "p.g": rnd(H * P, D)}
    h = rnd(T, D)
    rot = {"base": 30.0, "dims": dr, "scaling": {"factor": 4.0, "original": 32, "fast": 4.0, "slow": 0.5}}
    m = {"heads": H, "dim": d, "rot_dim": dr, "vdim": P, "kv_rank": R, "scale": 0.4, "rot": rot}
    got = latent_attention(h, w, "p.", m, 1e-4, torch.arange(T), None)
    f, amp = frequencies(dr, 30.0, rot["scaling"])
    assert amp > 1.1

    def turned(x, p):
        out = x.clone()
        for i in range(dr // 2):
            c, s = math.cos(p * f[i]) * amp, math.sin(p * f[i]) * amp
            out[i], out[i + dr // 2] = x[i] * c - x[i + dr // 2] * s, x[i + dr // 2] * c + x[i] * s
        return out
    rows = []
    for j in range(T):
        low = w["p.dkv"] @ h[j]
        c = low[:R] / torch.sqrt((low[:R] * low[:R]).mean() + 1e-4) * w["p.dkv.norm"]
        rows.append((c, turned(low[R:], j)))
    for i in range(T):
        for a in range(H):
            q = w["p.q"][a * (d + dr):(a + 1) * (d + dr)] @ h[i]
            qr = turned(q[d:], i)
            e = torch.stack([torch.exp(0.4 * (q[:d] @ (w["p.uk"][a * d:(a + 1) * d] @ c) + qr @ k)) for c, k in rows[:i + 1]])
            o = sum(e[j] * (w["p.uv"][a * P:(a + 1) * P] @ rows[j][0]) for j in range(i + 1)) / e.sum()
            assert torch.allclose(got[i, a * P:(a + 1) * P], o * torch.sigmoid(w["p.g"][a * P:(a + 1) * P] @ h[i]), atol=1e-6)


def test_routing_by_the_two_best_of_a_group():
    z = torch.tensor([[3.0, -4.0, 1.0, 0.9, 2.5, -3.0]])
    s = torch.sigmoid(z)[0]
    pick = lambda top, groups: choose_experts(z, top, groups)[0].tolist()
    assert pick(3, None) == [[0, 4, 2]]
    # groups (0 1) (2 3) (4 5): the best SUM of two is the second group's, though the largest score is in the first
    assert pick(2, (3, 1)) == [[2, 3]] and pick(2, (3, 2)) == [[4, 2]] and pick(3, (3, 3)) == [[0, 4, 2]]
    # groups of three: the third member has no say
    assert choose_experts(torch.tensor([[2.0, 1.0, 0.9, 2.1, 1.1, -9.0]]), 2, (2, 1))[0].tolist() == [[3, 4]]
    # groups of one expert: its score alone
    assert pick(2, (6, 3)) == [[0, 4]]
    D, E = 6, 6
    w = {"p.router": torch.eye(6)}
    for e in range(E):
        w.update({f"p.e{e}.up": torch.full((1, D), 0.5), f"p.e{e}.down": torch.full((D, 1), float(e + 1))})
    got = routed_ff(z, w, "p.", {"router": {"experts": E, "top": 2, "scale": 2.5, "groups": {"count": 3, "keep": 1}}}, None)
    act = float(gelu_erf(z.sum() * 0.5))
    want = 2.5 * (s[2] * 3 + s[3] * 4) / (s[2] + s[3]) * act
    assert torch.allclose(got, want.expand(1, D), atol=1e-5)
    w = {"p.gate": torch.eye(2), "p.gate.b": torch.tensor([0.5, 0.0]), "p.up": torch.eye(2), "p.up.b": torch.tensor([0.0, -1.0]),
         "p.down": 2.0 * torch.eye(2), "p.down.b": torch.tensor([0.1, 0.2])}
    h = torch.tensor([[1.0, 2.0]])
    assert torch.allclose(dense_ff(h, w, "p.", None), torch.stack([2 * silu(torch.tensor(1.5)) * 1.0 + 0.1, 2 * silu(torch.tensor(2.0)) * 1.0 + 0.2])[None])


def test_streams_are_read_and_written_from_the_old_ones():
    x = torch.tensor([[[1.0, 10.0], [2.0, 20.0]]])                       # one token, two streams of two values
    assert torch.allclose(read_streams(x, torch.tensor([3.0, -1.0])), torch.tensor([[1.0, 10.0]]))
    mix = torch.tensor([[0.5, 4.0], [2.0, -1.0]])                        # [from, to]
    y = torch.tensor([[7.0, 70.0]])
    got = write_streams(x, mix, torch.tensor([1.0, -2.0]), 0.1, y)
    assert torch.allclose(got, torch.tensor([[[0.5 + 4.0 + 0.7, 5.0 + 40.0 + 7.0], [4.0 - 2.0 - 1.4, 40.0 - 20.0 - 14.0]]]))
    h, w = torch.tensor([[1.0, -1.0]]), {"g": torch.tensor([[0.0, 1.0], [2.0, 0.0]]), "g.b": torch.tensor([1.0, -2.0])}
    assert torch.allclose(gated(y, h, w, "g", None), torch.tensor([[3.5, 35.0]]))


# ----------------------------------------------------------------------------- the engine's host logic
@pytest.mark.parametrize("name,cfg,page", [("A", TINY_A, 16), ("B", TINY_B, 8), ("M", ONLY_MEMORY, 32), ("T", ONLY_ATTENTION, 4), ("L", ONLY_LATENT, 16),
                                           ("P", ONE_PASS, 16)])
def test_host_logic_replay_cpu(tmp_path, name, cfg, page):
    d = make_lopilix_dir(str(tmp_path / name), cfg, seed=3)
    replay_all_schedules(d, cfg, "float32", [30, 13, 41, 1, 9, 22], page, HostOps(), "cpu", tail=8)


def test_greedy_generation_through_the_scheduler(tmp_path):
    d = make_lopilix_dir(str(tmp_path / "m"), TINY_A, seed=5)
    llm = LLM(d, dtype="float32", page_size=16, max_cached_tokens=512, max_num_seqs=4, max_num_batched_tokens=64,
              prefill_chunk=40, max_model_len=256, device="cpu", ops=HostOps(), use_cuda_graphs=False)
    prompts = [random_ids(n, TINY_A["vocab"], i) for i, n in enumerate([1, 5, 50, 33, 7])]
    outs = llm.generate(prompts, SamplingParams(greedy=True), max_tokens=4, eos_token_id=None)
    plain = PlainLopilix(d)
    for p, o in zip(prompts, outs):
        assert o.token_ids == greedy_by_the_plain_model(plain, p, 4)
    llm.engine.cache.check_invariants()
    assert not llm.engine.cache.requests and llm.scheduler.all_done()


def test_no_request_runs_past_the_position_table(tmp_path):
    """The learned positions end at max_positions: the last one is served, a longer request is refused before anything runs."""
    from llmengine_b200.config import EngineConfig
    from llmengine_b200.engine.engine import Engine, StepEntry, StepError
    d = make_lopilix_dir(str(tmp_path / "m"), ONE_PASS, seed=2)
    n = ONE_PASS["max_positions"]
    ec = EngineConfig(dtype="float32", max_cached_tokens=4 * n, max_num_seqs=2, max_num_batched_tokens=2 * n, device="cpu", use_cuda_graphs=False)
    eng = Engine(d, engine_config=ec, ops=HostOps())
    ids = random_ids(n, ONE_PASS["vocab"], 1)
    got = eng.step([StepEntry("a", ids, [n - 1])])
    assert float((got[0] - PlainLopilix(d).logits(ids)[-1]).abs().max()) < 1e-3
    with pytest.raises(StepError, match=str(n)):
        eng.step([StepEntry("a", [1], [0])])
    with pytest.raises(StepError, match=str(n)):
        eng.step([StepEntry("b", ids + [1], [n])])


def test_a_weight_file_that_does_not_fit_is_refused(tmp_path):
    from llmengine_b200.config import EngineConfig
    from llmengine_b200.engine.engine import Engine
    from llmengine_b200.weights import WeightError

    def damage(t):
        del t["l0.mix.lower"]
        t["l1.hc2.mix"] = t["l1.hc2.mix"][:-1].contiguous()
        t["l1.mix.lq3"] = torch.zeros(32, dtype=torch.bfloat16)
    d = make_lopilix_dir(str(tmp_path / "m"), TINY_A, seed=1, change=damage)
    ec = EngineConfig(dtype="float32", max_cached_tokens=64, max_num_seqs=2, max_num_batched_tokens=64, max_model_len=64, device="cpu")
    with pytest.raises(WeightError, match="l0.mix.lower") as e:
        Engine(d, engine_config=ec, ops=HostOps())
    assert "l1.hc2.mix" in str(e.value) and "l1.mix.lq3" in str(e.value)

    def unused(t):                                  # what belongs to a feed-forward sublayer that the layer lacks: ignored
        for n, shape in (("norm2", (50,)), ("hc2.in", (1,)), ("hc2.out", (1,)), ("hc2.mix", (1, 1)), ("rg2", (50, 50)), ("rg2.b", (50,))):
            t["l2." + n] = torch.zeros(shape, dtype=torch.bfloat16)
    d = make_lopilix_dir(str(tmp_path / "u"), TINY_B, seed=1, change=unused)
    Engine(d, engine_config=ec, ops=HostOps())
