"""Zuzupel without a device: configuration, registry, declared tensors, cache needs, chunk groups of the cache manager, the
plain implementation's own properties (one per mechanism), and the engine's host side (pages that chunks give back, slots with
the recurrences' state, layers that share weights, every cut) on the stand-in kernels."""
import json
import math

import numpy as np
import pytest
import torch

import plain_zuzupel as P
import replay_patterns as R
from cpu_ops import CpuOps
from zuzupel_configs import CONFIGS, L, delta, pair, random_weights, tokens, wkv
from bitwise_b200 import Model
from bitwise_b200.cache.manager import FREED, CacheManager, GroupSpec, groups_from_needs
from bitwise_b200.config import ConfigError, architecture_of
from bitwise_b200.config.zuzupel import ZuzupelConfig
from bitwise_b200.models.zuzupel import build_zuzupel
from bitwise_b200.parts import HalfRotaryEncoding, LinearScaling, PagedKVNeed, SlotStateNeed

F64 = torch.float64


def without_ranks(cfg):
    """The configuration as config.json gives it: the low ranks are tensors' shapes."""
    return ZuzupelConfig.from_json(cfg.to_json())


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_round_trip_registry_and_tensor_shapes(name):
    cfg = CONFIGS[name]
    raw = json.loads(json.dumps(cfg.to_json()))
    assert raw["architecture"] == "Zuzupel"
    arch = architecture_of(raw)
    assert arch.name == "Zuzupel"
    read = arch.config_from_json(raw)
    assert read.to_json() == cfg.to_json()
    shapes = {k: tuple(v.shape) for k, v in random_weights(cfg, 1).items()}
    assert read.with_tensor_shapes(shapes) == cfg


def test_config_optional_keys_and_errors():
    base = CONFIGS["a"].to_json()
    d = json.loads(json.dumps(base))
    left = d["layers"][0]["mixer"]["left"]
    left.pop("mask"), left["rot"].pop("scaling")
    c = ZuzupelConfig.from_json(d).layers[0].mixer.left
    assert c.chunk is None and c.rot_factor is None and c.rot_dims == 32
    left.pop("rot")
    assert ZuzupelConfig.from_json(d).layers[0].mixer.left.rot_dims is None
    for change, word in [(lambda d: d["layers"][2]["mixer"].update(kv_heads=4), "multiple"),
                         (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
                         (lambda d: d["layers"][1].update(type="other"), "unknown type"),
                         (lambda d: d["layers"][0]["mlp"].update(kind="moe"), "not supported"),
                         (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=34), "rot.dims"),
                         (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("factor"), "factor"),
                         (lambda d: d["layers"][0]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
                         (lambda d: d["layers"][0]["mixer"]["left"]["mask"].update(size=0), "mask.size"),
                         (lambda d: d["layers"][2]["mixer"].pop("conv"), "conv"),
                         (lambda d: d["layers"][4].update(weights_of=9), "no other layer"),
                         (lambda d: d["layers"][4].update(weights_of=4), "no other layer"),
                         (lambda d: d["layers"][2].update(weights_of=4), "no other layer"),   # a circle
                         (lambda d: d["layers"][4].update(weights_of=1), "differ"),
                         (lambda d: d["norm"].pop("eps"), "eps"),
                         (lambda d: d.pop("width"), "width")]:
        d = json.loads(json.dumps(base))
        change(d)
        with pytest.raises(ConfigError, match=word):
            ZuzupelConfig.from_json(d)
    d = json.loads(json.dumps(base))
    d["layers"].append(dict(d["layers"][4], weights_of=4))        # of a layer that itself uses another's
    assert ZuzupelConfig.from_json(d).owner(5) == 2


def test_declared_tensors_schedule_and_cache_needs():
    cfg = CONFIGS["a"]
    model = build_zuzupel(cfg)
    specs = {s.name: tuple(s.shape) for s in model.param_specs()}
    assert specs["embed"] == (149, 64) and specs["head"] == (149, 64) and specs["final.norm"] == (64,)
    assert specs["l0.mix.left.q"] == (128, 64) and specs["l0.mix.left.k.b"] == (64,) and specs["l0.mix.left.q.norm"] == (32,)
    assert specs["l0.mix.right.i"] == (2, 64) and specs["l0.mix.right.f.b"] == (2,) and specs["l0.mix.right.norm"] == (80,)
    assert specs["l0.mix.left.out"] == (64,) and specs["l0.mix.right.o"] == (64, 80) and "l0.mix.left.v.norm" not in specs
    assert specs["l1.mix.mu.w"] == (64,) and specs["l1.mix.w1"] == (10, 64) and specs["l1.mix.w2"] == (72, 10)
    assert specs["l1.mix.u"] == (3, 24) and specs["l1.mix.w0"] == (72,) and specs["l1.mix.g"] == (72, 64)
    assert specs["l2.mix.q"] == (32, 64) and specs["l2.mix.v.conv"] == (192, 3) and specs["l2.mix.a2"] == (96, 9)
    assert specs["l2.mix.A_log"] == (6,) and specs["l2.mix.norm"] == (32,) and specs["l2.mix.g2"] == (192, 20)
    assert "l2.norm2" not in specs and "l2.mlp.up" not in specs and specs["l0.mlp.down"] == (64, 112) and "l0.mlp.gate" not in specs
    assert not any(n.startswith("l4.") for n in specs)              # the last layer has no tensors of its own
    assert [r.block for r in model.schedule] == [0, 1, 2, 3, 2]
    f32 = torch.float32
    assert model.cache_needs() == [
        PagedKVNeed(2, 32, None, v_dim=16, chunk=40), SlotStateNeed((2, 41, 28), f32),
        SlotStateNeed((3, 24, 24), f32), SlotStateNeed((1, 64), f32),
        SlotStateNeed((6, 32, 16), f32), SlotStateNeed((2, 32 + 32 + 192), f32),
        PagedKVNeed(1, 16, None, v_dim=48, chunk=16), SlotStateNeed((1, 17, 44), f32),
        SlotStateNeed((6, 32, 16), f32), SlotStateNeed((2, 32 + 32 + 192), f32)]
    assert [(g.chunk, g.window, g.entries) for g in groups_from_needs(model.cache_needs())] == [(16, None, (6,)), (40, None, (0,))]
    # one tap keeps no inputs
    assert build_zuzupel(CONFIGS["b"]).cache_needs()[:2] == [SlotStateNeed((1, 5, 7), f32), SlotStateNeed((5, 9, 9), f32)]
    # a layer may use the weights of a later one
    names = {s.name for s in build_zuzupel(CONFIGS["c"]).param_specs()}
    assert "l3.mix.r" in names and not any(n.startswith("l1.") for n in names)
    assert not groups_from_needs(build_zuzupel(CONFIGS["d"]).cache_needs())


def test_stacked_projections_keep_every_weight():
    cfg = CONFIGS["b"]
    W = random_weights(cfg, 1)
    m = Model.from_tensors(cfg, W, dtype="float32", device="cpu", ops=CpuOps("float32"))
    d = m.decoder.blocks[0].mixer
    assert torch.equal(d.w_in[7:14], W["l0.mix.k"].float()) and torch.equal(d.w_in[d.low0:d.low0 + 3], W["l0.mix.a1"].float())
    assert torch.equal(d.w_in[d.beta0:d.beta0 + 1], W["l0.mix.b"].float()) and d.w_in.shape[0] % 8 == 0
    assert torch.equal(d.w_low[:7, :3], W["l0.mix.a2"].float()) and float(d.w_low[:7, 3:].abs().max()) == 0.0
    p = m.decoder.blocks[2].mixer
    assert torch.equal(p.left.w_in, torch.cat([W[f"l2.mix.left.{n}"] for n in "qkv"]).float())
    assert torch.equal(p.right.w_in[:30], W["l2.mix.right.q"].float()) and p.left_cols % 8 == 0


@pytest.mark.parametrize("page,size", [(16, 40), (16, 16), (4, 7), (8, 64), (16, 5)])
def test_chunk_groups_give_pages_back_at_a_chunk_end(page, size):
    mgr = CacheManager([GroupSpec(None, (0,)), GroupSpec(None, (1,), 0, size)], [64, 64], page, 2)
    mgr.begin("r")
    g = np.random.default_rng(size)
    length = 0
    while length < 200:
        new = length + int(g.integers(1, 23))
        assert mgr.ensure("r", new)
        mgr.advance("r", new)
        length = new
        tables = mgr.get("r").tables
        assert all(p != FREED for p in tables[0])
        first = length // size * size                              # the next position sees keys from here on
        for b, p in enumerate(tables[1]):
            assert (p == FREED) == ((b + 1) * page <= first), (length, b)
        mgr.check_consistency()
    mgr.release("r")
    assert mgr.all_free()


@pytest.mark.parametrize("dims,base,factor", [(8, 100.0, 4.0), (32, 5000.0, None), (10, 777.0, 1.0), (2, 20.0, 0.5)])
def test_rotary_tables_with_divided_frequencies(dims, base, factor):
    rot = {"dims": dims, "base": base}
    if factor:
        rot["scaling"] = {"factor": factor}
    enc = HalfRotaryEncoding(dims, base, LinearScaling(factor) if factor else None, positions=50)
    enc.reserve(300)                                              # grown in two pieces
    f = P.rotary_frequencies(rot)
    assert np.allclose(enc.freq64, f, rtol=1e-13)
    p = np.arange(300)[:, None]
    assert np.abs(enc._cos - np.cos(p * np.array(f))).max() < 1e-6 and np.abs(enc._sin - np.sin(p * np.array(f))).max() < 1e-6


def test_plain_recurrences_in_closed_form():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    n, H, d, v = 7, 2, 5, 3
    q, k, val = r(n, H, d), r(n, H, d), r(n, H, v)
    w = torch.rand(n, H, d, generator=g, dtype=F64)
    # bonus form: o_t = sum_(s < t) (r_t . (prod_(s < j < t) w_j) k_s) v_s + (r_t . u k_t) v_t
    u = r(H, d)
    o, _ = P.bonus_scan(q, k, val, w, u)
    for t in range(n):
        want = (q[t] * u * k[t]).sum(-1, keepdim=True) * val[t]
        for s in range(t):
            want = want + (q[t] * w[s + 1:t].prod(0) * k[s]).sum(-1, keepdim=True) * val[s]
        assert torch.allclose(o[t], want)
    # delta rule with a unit key, beta 1 and no decay: the value at that key is replaced
    e = torch.zeros(n, H, d, dtype=F64)
    e[:, :, 1] = 1.0
    o, S = P.delta_scan(e, e, val, torch.ones(n, H, d, dtype=F64), torch.ones(n, H, dtype=F64))
    assert torch.allclose(o, val) and torch.allclose(S[:, 1], val[-1])
    # ... and the old one is decayed before it is compared
    half = torch.full((n, H, d), 0.5, dtype=F64)
    o, _ = P.delta_scan(e, e, val, half, torch.full((n, H), 0.25, dtype=F64))
    assert torch.allclose(o[1], 0.5 * o[0] + 0.25 * (val[1] - 0.5 * o[0]))
    # matrix memory: the running maximum changes nothing where the denominator is the normaliser's
    i, f = r(n, H), -torch.rand(n, H, generator=g, dtype=F64)
    o, (S, nrm, m) = P.matrix_memory_scan(q, k, val, i, f)
    for t in range(n):
        num, den = torch.zeros(H, v, dtype=F64), torch.zeros(H, dtype=F64)
        mt = torch.stack([torch.zeros(H, dtype=F64) + f[:t + 1].sum(0)] + [i[s] + f[s + 1:t + 1].sum(0) for s in range(t + 1)]).max(0).values
        for s in range(t + 1):
            a = torch.exp(i[s] + f[s + 1:t + 1].sum(0)) * (q[t] * k[s]).sum(-1)
            num, den = num + a[:, None] * val[s], den + a
        den = torch.maximum((den * torch.exp(-mt)).abs(), torch.exp(-mt)) + 1e-6
        assert torch.allclose(o[t], num * torch.exp(-mt)[:, None] / den[:, None])
    # the state handed on gives the same as one walk
    a, st = P.matrix_memory_scan(q[:3], k[:3], val[:3], i[:3], f[:3])
    b, _ = P.matrix_memory_scan(q[3:], k[3:], val[3:], i[3:], f[3:], *st)
    assert torch.allclose(torch.cat([a, b]), o)


def test_plain_small_mechanisms():
    g = torch.Generator().manual_seed(1)
    u, w = torch.randn(6, 3, generator=g, dtype=F64), torch.randn(3, 4, generator=g, dtype=F64)
    y = P.causal_conv(u, w)
    assert torch.allclose(y[0], w[:, 3] * u[0])                                     # zeros before the start
    assert torch.allclose(y[5], w[:, 0] * u[2] + w[:, 1] * u[3] + w[:, 2] * u[4] + w[:, 3] * u[5])
    assert torch.allclose(P.causal_conv(u[:2], w)[1], w[:, 2] * u[0] + w[:, 3] * u[1])
    prev = P.previous_rows(u)
    assert float(prev[0].abs().max()) == 0.0 and torch.equal(prev[1:], u[:-1])
    seen = P.chunk_visible(range(10), 4)
    assert seen[7].nonzero().flatten().tolist() == [4, 5, 6, 7] and seen[8].nonzero().flatten().tolist() == [8]
    assert P.chunk_visible(range(10), None)[7].sum() == 8
    x = torch.randn(4, 8, generator=g, dtype=F64)
    assert torch.allclose(P.unit_length(x).norm(dim=-1), torch.ones(4, dtype=F64), atol=1e-5)
    ln = P.layer_norm(x, torch.ones(8, dtype=F64), 1e-9)
    assert torch.allclose(ln.mean(-1), torch.zeros(4, dtype=F64), atol=1e-12) and torch.allclose(ln.var(-1, unbiased=False), torch.ones(4, dtype=F64))
    assert math.isclose(float(P.softplus(torch.tensor(0.0, dtype=F64))), math.log(2.0))
    assert math.isclose(float(P.log_sigmoid(torch.tensor(-3.0, dtype=F64))), -math.log1p(math.exp(3.0)))
    v = torch.randn(9, 3, 12, generator=g, dtype=F64)
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 4.0}}
    out = P.rotate_half(v, range(20, 29), rot)
    assert torch.equal(out[..., 8:], v[..., 8:])                                    # entries beyond dims pass
    slow = P.rotate_half(v, [p / 4.0 for p in range(20, 29)], {"dims": 8, "base": 100.0})
    assert torch.allclose(out, slow)                                                # positions count a quarter
    for i in range(4):                                                              # pair i is (i, i + 4): lengths stay
        assert torch.allclose(out[..., i] ** 2 + out[..., i + 4] ** 2, v[..., i] ** 2 + v[..., i + 4] ** 2)


def test_plain_forward_is_causal_and_uses_every_tensor():
    for name in ("a", "b"):
        cfg = CONFIGS[name]
        W = {k: v.to(F64) for k, v in random_weights(cfg, 3).items()}
        toks = tokens(cfg, 50, 1)
        raw = cfg.to_json()
        full = P.forward(raw, W, toks)
        assert torch.allclose(full[:31], P.forward(raw, W, toks[:31]))             # later tokens change nothing earlier
        for n in W:
            W2 = dict(W)
            W2[n] = W[n] + 0.3 * torch.arange(1, W[n].numel() + 1, dtype=F64).cos().reshape(W[n].shape)
            assert not torch.allclose(full, P.forward(raw, W2, toks)), n


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cut_on_the_stand_in(name):
    cfg = CONFIGS[name]
    W = random_weights(cfg, 3)
    model = Model.from_tensors(cfg, W, dtype="float32", device="cpu", ops=CpuOps("float32"))
    reqs = {f"{name}{i}": tokens(cfg, n, i) for i, n in enumerate([37, 70, 5, 1, 18])}
    want = {rid: P.forward(cfg.to_json(), W, t).numpy() for rid, t in reqs.items()}
    for steps, pool in ((R.whole(reqs), 128), (R.tail_one_by_one(reqs, 9), 128), (R.portions(reqs, sizes=(3, 2, 11, 1)), 128),
                        (R.portions(reqs, sizes=(2,)), 128), (R.mixed(reqs, 192, seed=5), 192)):
        got = R.collect(steps, R.run_in_process(model, steps, pool), cfg.vocab)
        for rid in reqs:
            err = np.abs(got[rid] - want[rid]).max() / np.abs(want[rid]).max()
            assert err < 2e-4, (rid, err)


def test_chunk_layers_give_pages_back_through_the_stepper():
    from bitwise_b200.engine.replay import make_replay_stepper
    from bitwise_b200.engine.step import StepEntry
    cfg = CONFIGS["a"]
    model = Model.from_tensors(cfg, random_weights(cfg, 3), dtype="float32", device="cpu", ops=CpuOps("float32"))
    stepper = make_replay_stepper(model, 256, 16, max_live=2)
    stepper.run([StepEntry("r", tokens(cfg, 150, 4), [149])])
    groups = stepper.manager.groups
    tables = stepper.manager.get("r").tables
    held = {g.chunk: sum(1 for p in tables[i] if p != FREED) for i, g in enumerate(groups)}
    assert held == {16: 1, 40: 3}                                   # positions from 144, from 120 on
    stepper.finish("r")
    assert stepper.manager.all_free()


def test_greedy_generation_through_the_engine_on_the_stand_in():
    from bitwise_b200 import Engine, EngineConfig, SamplingParams
    cfg = CONFIGS["d"]                                              # no pages: admission by slots and budget alone
    W = random_weights(cfg, 3)
    model = Model.from_tensors(cfg, W, dtype="float32", device="cpu", ops=CpuOps("float32"))
    prompts = [tokens(cfg, n, 200 + i) for i, n in enumerate([5, 40, 1])]
    got = Engine(model, EngineConfig(num_blocks=12, block_size=16, max_batched_tokens=16, max_num_seqs=2)).generate(
        prompts, SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True))
    for prompt, out in zip(prompts, got):
        seq = list(prompt)
        for t in out:
            row = P.forward(cfg.to_json(), W, seq)[-1].numpy()
            assert t == int(row.argmax()) or row.max() - row[t] < 1e-4 * np.abs(row).max()
            seq.append(t)


def test_folder_round_trip(tmp_path):
    import os
    from bitwise_b200.weights.safetensors_io import SafetensorsFile
    cfg = CONFIGS["b"]
    folder = Model.write_random_folder(str(tmp_path / "m"), cfg, seed=4, std=0.3, norm_jitter=0.2)
    stored = json.load(open(os.path.join(folder, "config.json")))
    assert {k: v for k, v in stored.items() if k != "torch_dtype"} == cfg.to_json()
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    tensors = {n: f.tensor(n).clone() for n in f.names()}
    assert tuple(tensors["l0.mix.a1"].shape) == (3, 50)
    toks = tokens(cfg, 40, 2)
    got = Model.load(folder, "float32", device="cpu", ops=CpuOps("float32")).logits(toks)
    want = P.forward(stored, tensors, toks).numpy()
    assert np.abs(got - want).max() < 2e-4 * np.abs(want).max()
