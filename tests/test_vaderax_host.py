"""The Vaderax design on the host: configuration, the order of a loop, tensor names, the cache a layer asks for, the plain
implementation's mechanisms on inputs whose result can be written down, and the engine's own logic (batch metadata, pages,
state slots, scheduling) with a CPU stand-in for the kernels, against the plain implementation."""
import copy
import math

import pytest
import torch

from helpers import random_ids
from host_ops import HostOps
from llmengine_b200 import LLM, SamplingParams
from llmengine_b200.config import ConfigError, VaderaxConfig, config_from_dict
from llmengine_b200.engine.model import Model
from llmengine_b200.parts import Runtime
from llmengine_b200.parts.base import StatesSpec
from plain_vaderax import (PlainVaderax, attention, choose_experts, causal_conv, delta_mixer, delta_rule, layer_norm, relu_squared,
                           rotate_half, routed_ff, runs, silu, softplus, unit_rms, unit_vector)
from tiny_vaderax import ONE_PASS, ONLY_ATTENTION, ONLY_DELTA, TINY_A, TINY_B, make_vaderax_dir, tensor_shapes
from vaderax_cases import greedy_by_the_plain_model, replay_all_schedules

ALL = [("A", TINY_A), ("B", TINY_B), ("D", ONLY_DELTA), ("T", ONLY_ATTENTION), ("P", ONE_PASS)]


def test_every_size_and_constant_comes_from_the_file():
    c = config_from_dict(TINY_A)
    assert isinstance(c, VaderaxConfig) and (c.hidden_size, c.vocab_size, c.norm_eps, c.embedding_scale) == (64, 103, 1e-5, 7.0)
    d, a = c.mixers[0], c.mixers[1]
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.taps) == (4, 2, 16, 32, 4)
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.rot_base, a.rot_dims) == (4, 2, 32, 32, 0.2, 500.0, 16)
    f = c.mlps
    assert (f[0].kind, f[0].ff) == ("dense", 96) and f[3] is None
    assert (f[1].ff, f[1].experts, f[1].top, f[1].identity, f[1].groups, f[1].keep) == (24, 7, 3, 2, 3, 2)
    b = config_from_dict(TINY_B)
    assert (b.mlps[1].identity, b.mlps[1].groups, b.mlps[1].keep) == (0, 1, 1)
    for _, cfg in ALL:
        assert config_from_dict(config_from_dict(cfg).to_dict()) == config_from_dict(cfg)
    for path in (["width"], ["norm"], ["embedding", "scale"], ["layers", 0, "mixer", "vdim"], ["layers", 0, "mixer", "conv"],
                 ["layers", 0, "mixer", "kv_heads"], ["layers", 1, "mixer", "scale"], ["layers", 1, "mixer", "rot", "base"],
                 ["layers", 1, "mixer", "rot", "dims"], ["layers", 1, "mlp", "router", "top"], ["layers", 1, "mlp", "expert"],
                 ["layers", 1, "mlp", "router", "groups", "keep"], ["layers", 0, "mlp", "ff"], ["layers", 2, "type"], ["loop", "times"]):
        e = copy.deepcopy(TINY_A)
        at = e
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=str(path[-1])):
            config_from_dict(e)
    for edit, word in ((lambda e: e["layers"][0]["mixer"].__setitem__("kv_heads", 3), "kv_heads"),
                       (lambda e: e["layers"][1]["mixer"]["rot"].__setitem__("dims", 34), "rot.dims"),
                       (lambda e: e["layers"][1]["mlp"]["router"].__setitem__("top", 7), "top"),
                       (lambda e: e["layers"][1]["mlp"]["router"]["groups"].__setitem__("count", 4), "count"),
                       (lambda e: e["layers"][1]["mlp"]["router"]["groups"].__setitem__("keep", 4), "keep"),
                       (lambda e: e["loop"].__setitem__("stop", 5), "loop.stop"),
                       (lambda e: e["layers"][0].__setitem__("type", "something_else"), "something_else"),
                       (lambda e: e["layers"][0]["mlp"].__setitem__("kind", "sparse"), "sparse")):
        e = copy.deepcopy(TINY_A)
        edit(e)
        with pytest.raises(ConfigError, match=word):
            config_from_dict(e)


def test_the_order_of_a_loop():
    """Every pass over the looped layers is a run of its own (with a cache of its own); the embedding output is added right before
    the first layer of every pass but the first, and nowhere else."""
    order = lambda cfg: [(r.layer, r.add_embedding) for r in config_from_dict(cfg).model_spec().order]
    assert order(TINY_A) == [(0, False), (1, False), (0, True), (1, False), (0, True), (1, False), (2, False), (3, False)]
    assert order(TINY_B) == [(0, False), (1, False), (1, True), (2, False), (3, False)]
    assert order(ONLY_DELTA) == [(0, False), (1, False), (1, True), (1, True)]
    assert order(ONE_PASS) == [(0, False), (1, False)]
    no_loop = {k: v for k, v in TINY_A.items() if k != "loop"}
    assert order(no_loop) == [(i, False) for i in range(4)]
    empty = dict(TINY_A, loop={"start": 2, "stop": 2, "times": 3})
    assert order(empty) == order(no_loop)
    for _, cfg in ALL:
        assert order(cfg) == runs(cfg)
    spec = config_from_dict(TINY_A).model_spec()
    assert all(r.cache_from is None for r in spec.order)


@pytest.mark.parametrize("name,cfg", ALL)
def test_the_model_declares_the_design_s_tensors(name, cfg):
    m = Model(config_from_dict(cfg).model_spec(), Runtime(None, torch.device("cpu"), torch.float32, 1))
    assert {n: tuple(s.shape) for n, s in m.weight_specs().items()} == tensor_shapes(cfg)


def test_what_each_layer_keeps_between_steps():
    m = Model(config_from_dict(TINY_A).model_spec(), Runtime(None, torch.device("cpu"), torch.float32, 1))
    specs = [b.cache_spec() for b in m.blocks]
    assert isinstance(specs[0], StatesSpec) and dict(specs[0].parts) == {"conv": (3, 2 * 2 * 16 + 4 * 32), "state": (4, 32, 16)}
    assert specs[1].paged and specs[1].window == 0 and (specs[3].k_dim, specs[3].v_dim) == (16, 48)
    assert len(m.cache_specs()) == 8, "every pass of the loop keeps a cache of its own"


# ----------------------------------------------------------------------------- the plain implementation against itself
def test_plain_mechanisms_by_hand():
    x = torch.tensor([[3.0, 4.0]])
    assert torch.allclose(unit_rms(x, 0.0), x / (12.5 ** 0.5)) and torch.allclose(unit_vector(x, 0.0), x / 5.0)
    assert torch.allclose(layer_norm(torch.tensor([[1.0, 3.0]]), torch.tensor([2.0, 5.0]), torch.tensor([0.5, 7.0]), 0.0), torch.tensor([[-1.5, 12.0]]))
    assert relu_squared(torch.tensor([-2.0, 3.0])).tolist() == [0.0, 9.0]
    assert abs(float(softplus(torch.tensor(0.0))) - math.log(2.0)) < 1e-6 and abs(float(silu(torch.tensor(1.0))) - 0.7310586) < 1e-6
    # the last column of the taps meets the present token; zeros before the start
    y = causal_conv(torch.tensor([[1.0], [10.0], [100.0]]), torch.tensor([[2.0, 3.0, 5.0]]))
    assert y.view(-1).tolist() == [5 * 1, 5 * 10 + 3 * 1, 5 * 100 + 3 * 10 + 2 * 1]
    # rotation: position 0 changes nothing; coordinates from `dims` on pass; i pairs with i + dims/2; pair 0 has frequency 1
    v = torch.arange(12.0).view(1, 2, 6)
    assert torch.equal(rotate_half(v, torch.tensor([0]), 100.0, 4), v)
    r = rotate_half(v.expand(3, 2, 6), torch.tensor([0, 1, 7]), 100.0, 4)
    assert torch.equal(r[..., 4:], v.expand(3, 2, 6)[..., 4:])
    c, s = math.cos(7.0), math.sin(7.0)
    assert abs(float(r[2, 0, 0]) - (0 * c - 2 * s)) < 1e-5 and abs(float(r[2, 0, 2]) - (2 * c + 0 * s)) < 1e-5
    c, s = math.cos(7.0 * 100.0 ** -0.5), math.sin(7.0 * 100.0 ** -0.5)
    assert abs(float(r[2, 1, 1]) - (7 * c - 9 * s)) < 1e-5 and abs(float(r[2, 1, 3]) - (9 * c + 7 * s)) < 1e-5


def test_the_delta_rule_is_a_product_of_transitions():
    """S_t = a_t (1 - b_t k k^T) S_(t-1) + b_t k v^T, written out as matrices; with unit keys and b = 1, a = 1 a key that comes
    again finds exactly the value last written under it; handing the state on at a cut changes nothing."""
    g = torch.Generator().manual_seed(0)
    T, d, P = 6, 4, 3
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v = rnd(T, 1, d), unit_vector(rnd(T, 1, d), 0.0), rnd(T, 1, P)
    beta, keep = torch.sigmoid(rnd(T, 1)), torch.sigmoid(rnd(T, 1))
    o, S = delta_rule(q, k, v, beta, keep)
    M = torch.zeros(d, P, dtype=torch.float64)
    for t in range(T):
        kt = k[t, 0]
        M = keep[t, 0] * (torch.eye(d, dtype=torch.float64) - beta[t, 0] * torch.outer(kt, kt)) @ M + beta[t, 0] * torch.outer(kt, v[t, 0])
        assert torch.allclose(o[t, 0], M.t() @ q[t, 0], atol=1e-12)
    first, S1 = delta_rule(q[:2], k[:2], v[:2], beta[:2], keep[:2])
    second, S2 = delta_rule(q[2:], k[2:], v[2:], beta[2:], keep[2:], S1)
    assert torch.allclose(torch.cat([first, second]), o) and torch.allclose(S2, S)
    k[1] = k[0]
    one = torch.ones(2, 1, dtype=torch.float64)
    o, _ = delta_rule(k[:2], k[:2], v[:2], one, one)
    assert torch.allclose(o[0], v[0]) and torch.allclose(o[1], v[1]), "the second write replaces the first"


def test_the_delta_mixer_written_out():
    """Two value heads on one query/key head, two taps, every projection a selection of the input's coordinates."""
    g = torch.Generator().manual_seed(1)
    T, H, G, d, P = 5, 2, 1, 3, 2
    D = 2 * G * d + 2 * H * P + 2 * H
    h = torch.randn(T, D, generator=g, dtype=torch.float64)
    eye = torch.eye(D, dtype=torch.float64)
    w, at = {}, 0
    for n, size in (("q", G * d), ("k", G * d), ("v", H * P), ("g", H * P), ("b", H), ("a", H)):
        w["p." + n] = eye[at:at + size]
        at += size
    for n, c in (("q", G * d), ("k", G * d), ("v", H * P)):
        w[f"p.{n}.conv"] = torch.randn(c, 2, generator=g, dtype=torch.float64)
    w.update({"p.A_log": torch.tensor([0.2, -0.7], dtype=torch.float64), "p.dt_bias": torch.tensor([0.1, -1.0], dtype=torch.float64),
              "p.norm": torch.tensor([1.5, 0.5], dtype=torch.float64)})
    got = delta_mixer(h, w, "p.", {"heads": H, "kv_heads": G, "dim": d, "vdim": P, "conv": 2}, 1e-5, None)
    act = lambda n, lo, hi, t: silu(h[t, lo:hi] * w[f"p.{n}.conv"][:, 1] + (h[t - 1, lo:hi] * w[f"p.{n}.conv"][:, 0] if t else 0.0))
    for x in range(H):
        S = torch.zeros(d, P, dtype=torch.float64)
        for t in range(T):
            q, k, v = act("q", 0, d, t), act("k", d, 2 * d, t), act("v", 2 * d, 2 * d + H * P, t)[x * P:(x + 1) * P]
            q, k = q / torch.sqrt((q * q).sum() + 1e-6) / math.sqrt(d), k / torch.sqrt((k * k).sum() + 1e-6)
            z = 2 * d + H * P
            gate, b, a = h[t, z + x * P:z + (x + 1) * P], h[t, z + H * P + x], h[t, z + H * P + H + x]
            S = torch.exp(-torch.exp(w["p.A_log"][x]) * torch.log1p(torch.exp(a + w["p.dt_bias"][x]))) * S
            S = S + torch.outer(k, torch.sigmoid(b) * (v - S.t() @ k))
            o = S.t() @ q
            o = o / torch.sqrt((o * o).mean() + 1e-5) * w["p.norm"] * gate * torch.sigmoid(gate)
            assert torch.allclose(got[t, x * P:(x + 1) * P], o, atol=1e-10)


def test_attention_written_out():
    """Two query heads on one key/value head, half of a head rotated, the norm behind the rotation, the gate on the heads."""
    g = torch.Generator().manual_seed(2)
    T, H, d, P, D = 5, 2, 4, 3, 6
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    w = {"p.q": rnd(H * d, D), "p.k": rnd(d, D), "p.v": rnd(P, D), "p.g": rnd(H * P, D)}
    h, pos = rnd(T, D), torch.arange(T)
    got = attention(h, w, "p.", {"heads": H, "kv_heads": 1, "dim": d, "vdim": P, "scale": 0.7, "rot": {"base": 20.0, "dims": 2}}, 1e-4, pos, None)

    def finished(x, p):
        u, v = float(x[0]), float(x[1])
        x = torch.cat([torch.tensor([u * math.cos(p) - v * math.sin(p), v * math.cos(p) + u * math.sin(p)], dtype=torch.float64), x[2:]])
        return x / torch.sqrt((x * x).mean() + 1e-4)
    keys, vals = [finished(w["p.k"] @ h[j], j) for j in range(T)], [w["p.v"] @ h[j] for j in range(T)]
    for i in range(T):
        for a in range(H):
            q = finished(w["p.q"][a * d:(a + 1) * d] @ h[i], i)
            e = torch.stack([torch.exp(0.7 * (q @ keys[j])) for j in range(i + 1)])
            o = sum(e[j] * vals[j] for j in range(i + 1)) / e.sum() * torch.sigmoid(w["p.g"][a * P:(a + 1) * P] @ h[i])
            assert torch.allclose(got[i, a * P:(a + 1) * P], o, atol=1e-6)


def test_routing_by_groups_with_corrections_and_identity_experts():
    z = torch.tensor([[2.0, 0.0, 1.9, 1.8, -1.0, 1.0]])
    s = torch.softmax(z, -1)[0]
    pick = lambda corr, top, groups: choose_experts(z, torch.tensor(corr), top, groups)[:2]
    idx, wt = pick([0.0] * 6, 3, None)
    assert idx.tolist() == [[0, 2, 3]] and torch.allclose(wt[0], s[[0, 2, 3]]), "the weights are not renormalised"
    # groups (0 1) (2 3) (4 5): only the first two groups offer their members
    assert pick([0.0] * 6, 2, (3, 1))[0].tolist() == [[0, 1]] and pick([0.0] * 6, 3, (3, 2))[0].tolist() == [[0, 2, 3]]
    # the choice goes by the corrected scores, the weights do not; negative choice scores are still ahead of what is not offered
    idx, wt = pick([0.0, 0.0, 0.0, 0.0, 0.0, 5.0], 2, (3, 1))
    assert idx.tolist() == [[5, 4]] and torch.allclose(wt[0], s[[5, 4]])
    idx, _ = pick([-3.0, -4.0, -6.0, -7.0, -8.0, -9.0], 2, (3, 1))
    assert idx.tolist() == [[0, 1]]
    # the last output of the router stands for the input
    D, E = 6, 5
    w = {"p.router": torch.eye(6), "p.correction": torch.zeros(6)}
    for e in range(E):
        w.update({f"p.e{e}.up": torch.full((1, D), 1.0), f"p.e{e}.down": torch.full((D, 1), float(e + 1))})
    h = z.clone()
    got = routed_ff(h, w, "p.", {"router": {"experts": E, "identity": 1, "top": 6, "groups": {"count": 2, "keep": 2}}}, None)
    up2 = float(h.sum()) ** 2
    want = sum(s[e] * (e + 1) for e in range(E)) * up2 + s[5] * h[0]
    assert torch.allclose(got[0], want, atol=1e-4)


# ----------------------------------------------------------------------------- the engine's host logic
@pytest.mark.parametrize("name,cfg,page", [("A", TINY_A, 16), ("B", TINY_B, 8), ("D", ONLY_DELTA, 32), ("T", ONLY_ATTENTION, 4), ("P", ONE_PASS, 16)])
def test_host_logic_replay_cpu(tmp_path, name, cfg, page):
    d = make_vaderax_dir(str(tmp_path / name), cfg, seed=3)
    replay_all_schedules(d, cfg, "float32", [30, 13, 41, 1, 9, 22], page, HostOps(), "cpu", tail=8)


def test_greedy_generation_through_the_scheduler(tmp_path):
    d = make_vaderax_dir(str(tmp_path / "m"), TINY_A, seed=5)
    llm = LLM(d, dtype="float32", page_size=16, max_cached_tokens=512, max_num_seqs=4, max_num_batched_tokens=64,
              prefill_chunk=40, max_model_len=256, device="cpu", ops=HostOps(), use_cuda_graphs=False)
    prompts = [random_ids(n, TINY_A["vocab"], i) for i, n in enumerate([1, 5, 50, 33, 7])]
    outs = llm.generate(prompts, SamplingParams(greedy=True), max_tokens=4, eos_token_id=None)
    plain = PlainVaderax(d)
    for p, o in zip(prompts, outs):
        assert o.token_ids == greedy_by_the_plain_model(plain, p, 4)
    llm.engine.cache.check_invariants()
    assert not llm.engine.cache.requests and llm.scheduler.all_done()


def test_a_weight_file_that_does_not_fit_is_refused(tmp_path):
    from llmengine_b200.config import EngineConfig
    from llmengine_b200.engine.engine import Engine
    from llmengine_b200.weights import WeightError

    def damage(t):
        del t["l0.mix.dt_bias"]
        t["l1.mlp.correction"] = t["l1.mlp.correction"][:-1].contiguous()
        t["l1.mlp.e7.up"] = torch.zeros(24, 64, dtype=torch.bfloat16)   # an identity expert has no tensors
        t["l3.norm2"] = t["l3.norm2.b"] = torch.zeros(64, dtype=torch.bfloat16)     # a norm for a feed-forward the layer lacks: ignored
    d = make_vaderax_dir(str(tmp_path / "m"), TINY_A, seed=1, change=damage)
    ec = EngineConfig(dtype="float32", max_cached_tokens=64, max_num_seqs=2, max_num_batched_tokens=64, max_model_len=64, device="cpu")
    with pytest.raises(WeightError, match="l0.mix.dt_bias") as e:
        Engine(d, engine_config=ec, ops=HostOps())
    assert "l1.mlp.correction" in str(e.value) and "l1.mlp.e7.up" in str(e.value) and "l3.norm2" not in str(e.value)
