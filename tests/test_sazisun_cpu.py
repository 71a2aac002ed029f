"""Sazisun without a device: configuration, registry, declared tensors, cache needs, the rotary tables, the plain
implementation's own properties (one per mechanism), and the engine's host side (pages that two layers read, slots with the state
and the convolution's inputs, every cut) on the stand-in kernels."""
import json
import math

import numpy as np
import pytest
import torch

import plain_sazisun as P
import replay_patterns as R
from cpu_ops import CpuOps
from sazisun_configs import CONFIGS, random_weights, tokens
from bitwise_b200 import Model
from bitwise_b200.cache.manager import groups_from_needs
from bitwise_b200.config import ConfigError, architecture_of
from bitwise_b200.config.sazisun import SazisunConfig
from bitwise_b200.models.sazisun import build_sazisun
from bitwise_b200.parts import PagedKVNeed, PairRotaryEncoding, SlotStateNeed, WavelengthScaling

F64 = torch.float64


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_round_trip_and_registry(name):
    cfg = CONFIGS[name]
    raw = json.loads(json.dumps(cfg.to_json()))
    assert raw["architecture"] == "Sazisun"
    arch = architecture_of(raw)
    assert arch.name == "Sazisun" and arch.config_from_json(raw) == cfg


def test_config_optional_keys_and_errors():
    base = CONFIGS["a"].to_json()
    d = json.loads(json.dumps(base))
    d["layers"] = d["layers"][:2]
    att, moe = d["layers"][0]["mixer"], d["layers"][1]["mlp"]
    att.pop("softcap"), att["rot"].pop("scaling"), moe.pop("shared"), moe["router"].pop("groups"), moe["router"].pop("scale")
    c = SazisunConfig.from_json(d)
    m, f = c.layers[0].mixer, c.layers[1].mlp
    assert m.softcap is None and m.rot_scaling is None and m.rot_dims == 8
    assert (f.groups, f.keep_groups, f.scale, f.shared_ff) == (1, 1, 1.0, None)
    att.pop("rot")
    d["layers"][0].pop("mlp")
    c = SazisunConfig.from_json(d)
    assert c.layers[0].mixer.rot_dims is None and c.layers[0].mlp is None
    for change, word in [(lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
                         (lambda d: d["layers"][1]["mixer"].update(groups=4), "multiple"),
                         (lambda d: d["layers"][1]["mixer"].update(norm_groups=5), "multiple"),
                         (lambda d: d["layers"][1].update(type="other"), "unknown type"),
                         (lambda d: d["layers"][0]["mlp"].update(kind="other"), "not supported"),
                         (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=18), "rot.dims"),
                         (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("low"), "low"),
                         (lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(low=7.0), "above"),
                         (lambda d: d["layers"][0]["mixer"].update(softcap=0), "softcap"),
                         (lambda d: d["layers"][0]["mixer"].pop("diff"), "diff"),
                         (lambda d: d["layers"][1]["mlp"]["router"].update(top=5), "choices"),
                         (lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=4), "multiple"),
                         (lambda d: d["layers"][2]["mixer"].update(kv_from=2), "earlier attention layer"),
                         (lambda d: d["layers"][2]["mixer"].update(kv_from=1), "earlier attention layer"),
                         (lambda d: d["layers"][2]["mixer"].update(dim=8), "differ"),
                         (lambda d: d["layers"][3]["mixer"].update(kv_from=2), "earlier attention layer"),
                         (lambda d: d["norm"].pop("eps"), "eps"),
                         (lambda d: d.pop("width"), "width")]:
        d = json.loads(json.dumps(base))
        change(d)
        with pytest.raises(ConfigError, match=word):
            SazisunConfig.from_json(d)


def test_declared_tensors_schedule_and_cache_needs():
    model = build_sazisun(CONFIGS["a"])
    specs = {s.name: tuple(s.shape) for s in model.param_specs()}
    assert specs["embed"] == (149, 80) and "head" not in specs and specs["final.norm.alpha"] == () and specs["final.norm.b"] == (80,)
    assert specs["l0.mix.q"] == (128, 80) and specs["l0.mix.k"] == (64, 80) and specs["l0.mix.v"] == (64, 80)
    assert specs["l0.mix.g"] == (128, 80) and specs["l0.mix.o"] == (80, 128) and specs["l0.mix.lk2"] == (16,)
    assert specs["l0.mlp.gate"] == (112, 80) and specs["l0.norm2.alpha"] == ()
    assert specs["l1.mix.in"] == (96 + 96 + 2 * 72 + 6, 80) and specs["l1.mix.conv"] == (240, 4) and specs["l1.mix.conv.b"] == (240,)
    assert specs["l1.mix.A_log"] == specs["l1.mix.dt_bias"] == specs["l1.mix.D"] == (6,) and specs["l1.mix.norm"] == (96,)
    assert specs["l1.mlp.e5.up"] == (24, 80) and "l1.mlp.e0.gate" not in specs and specs["l1.mlp.shared.sg"] == (1, 80)
    assert specs["l1.mlp.shared.down"] == (80, 40) and "l1.mlp.correction" not in specs
    assert "l2.mix.k" not in specs and "l2.mix.v" not in specs and specs["l2.mix.lq1"] == (16,) and "l2.norm2" not in specs
    assert "l3.mlp.shared.up" not in specs and "l3.mlp.shared.sg" not in specs
    f32 = torch.float32
    assert model.cache_needs() == [PagedKVNeed(4, 16, None, v_dim=32, v_heads=2), SlotStateNeed((6, 16, 24), f32), SlotStateNeed((3, 240), f32),
                                   PagedKVNeed(6, 32, None, v_dim=48, v_heads=3), SlotStateNeed((2, 32, 16), f32), SlotStateNeed((2, 96), f32)]
    assert [(r.cache, r.owns_cache, r.state) for r in model.schedule] == [(0, True, None), (1, True, 2), (0, False, None), (3, True, None), (4, True, 5)]
    assert build_sazisun(CONFIGS["b"]).schedule[0].state is None                       # one tap keeps no inputs
    assert [r.cache for r in build_sazisun(CONFIGS["c"]).schedule[1:4]] == [2, 2, 2]
    assert not groups_from_needs(build_sazisun(CONFIGS["d"]).cache_needs())


def test_stacked_weights_and_constants_made_at_load():
    cfg = CONFIGS["b"]
    W = random_weights(cfg, 1)
    m = Model.from_tensors(cfg, W, dtype="float32", device="cpu", ops=CpuOps("float32"))
    a, f = m.decoder.blocks[1].mixer, m.decoder.blocks[1].feed_forward
    assert torch.equal(a.w_in, torch.cat([W[f"l1.mix.{n}"] for n in "qkvg"]).float())
    want = P.subtraction_weight({k: v.to(F64) for k, v in W.items()}, "l1.mix.", 0.2)
    assert abs(float(a.lam) - float(want)) < 1e-6
    assert torch.equal(f.w_router[:5], W["l1.mlp.router"].float()) and torch.equal(f.w_router[5:6], W["l1.mlp.shared.sg"].float())
    assert f.w_gate_up.shape == (5, 9, 50) and torch.equal(f.w_gate_up[3], W["l1.mlp.e3.up"].float())
    s = m.decoder.blocks[0].mixer
    assert torch.allclose(s.rate.double(), W["l0.mix.A_log"].double().exp(), rtol=1e-6)
    with pytest.raises(NotImplementedError):
        type(a)(50, 4, 2, 8, 8, 0.3, difference=0.4, sink=True)


@pytest.mark.parametrize("dims,base,scaling", [(8, 100.0, None), (64, 5e5, (8.0, 1.0, 4.0, 8192)), (12, 700.0, (3.0, 2.0, 2.0, 60)), (32, 1e4, (2.5, 1.5, 9.0, 300)),
                                               (2, 20.0, (4.0, 1.0, 4.0, 4))])
def test_rotary_tables_with_rescaled_wavelengths(dims, base, scaling):
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    enc = PairRotaryEncoding(dims, base, WavelengthScaling(*scaling) if scaling else None, positions=50)
    enc.reserve(300)                                              # grown in two pieces
    f = P.rotary_frequencies(rot)
    assert enc.layout == "pairs" and np.allclose(enc.freq64, f, rtol=1e-13)
    p = np.arange(300)[:, None]
    assert np.abs(enc._cos - np.cos(p * np.array(f))).max() < 1e-6 and np.abs(enc._sin - np.sin(p * np.array(f))).max() < 1e-6
    if scaling and dims >= 32:                                    # all three ranges occur
        plain = np.array(P.rotary_frequencies({"dims": dims, "base": base}))
        ratio = np.array(f) / plain
        assert ratio[0] == 1.0 and math.isclose(ratio[-1], 1.0 / scaling[0]) and ((ratio < 0.999) & (ratio > 1.001 / scaling[0])).any()


def test_plain_mechanisms():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    # the recurrence in closed form: y_t = sum_(s <= t) prod_(s < j <= t) a_j (C_t . B_s) dt_s x_s + D x_t
    n, H, N, v = 7, 2, 5, 3
    x, B, C, dt, rate, D = r(n, H, v), r(n, H, N), r(n, H, N), torch.rand(n, H, generator=g, dtype=F64), torch.rand(H, generator=g, dtype=F64), r(H)
    y, S = P.space_scan(x, B, C, dt, rate, D)
    a = torch.exp(-rate * dt)
    for t in range(n):
        want = D[:, None] * x[t]
        for s in range(t + 1):
            want = want + (a[s + 1:t + 1].prod(0) * dt[s] * (C[t] * B[s]).sum(-1))[:, None] * x[s]
        assert torch.allclose(y[t], want)
    first, mid = P.space_scan(x[:3], B[:3], C[:3], dt[:3], rate, D)
    rest, end = P.space_scan(x[3:], B[3:], C[3:], dt[3:], rate, D, mid)
    assert torch.allclose(torch.cat([first, rest]), y) and torch.allclose(end, S)
    # convolution with a bias
    u, w, b = r(6, 3), r(3, 4), r(3)
    c = P.causal_conv(u, w, b)
    assert torch.allclose(c[0], b + w[:, 3] * u[0]) and torch.allclose(c[5], b + w[:, 0] * u[2] + w[:, 1] * u[3] + w[:, 2] * u[4] + w[:, 3] * u[5])
    # every part of a row by its own root mean square, the gate first
    o = P.gated_group_norm(r(4, 12), r(4, 12), torch.ones(12, dtype=F64), 3, 1e-12)
    assert torch.allclose(o.reshape(4, 3, 4).pow(2).mean(-1), torch.ones(4, 3, dtype=F64))
    # equal maps with lambda one leave nothing; lambda zero leaves the first map
    q, k, val = r(9, 2, 4), r(9, 2, 4), r(9, 2, 6)
    att = P.capped_attention(q, k, val, 0.5, 3.0)
    assert torch.allclose(att[0], val[0])                          # the first position sees itself alone
    assert float(P.subtract_and_norm(att, att, 1.0, 0.5, 1e-6).abs().max()) == 0.0
    assert torch.allclose(P.subtract_and_norm(att, q[..., :1] * val, 0.0, 0.25, 0.0), P.unit_rms(att, 0.0) * 0.75)
    s = (q[8, 0] * k[:, 0]).sum(-1) * 0.5
    assert torch.allclose(att[8, 0], (torch.softmax(3.0 * torch.tanh(s / 3.0), 0)[:, None] * val[:, 0]).sum(0))
    # rotation: pairs of neighbours keep their lengths, entries beyond dims pass
    t = r(9, 3, 12)
    rot = {"dims": 8, "base": 100.0}
    out = P.rotate_pairs(t, range(20, 29), rot)
    assert torch.equal(out[..., 8:], t[..., 8:])
    for i in range(4):
        assert torch.allclose(out[..., 2 * i] ** 2 + out[..., 2 * i + 1] ** 2, t[..., 2 * i] ** 2 + t[..., 2 * i + 1] ** 2)
    # the choice: only the groups with the largest scores; weights over their sum
    z = torch.tensor([3.0, 0.0, 2.5, 2.4, 1.0, 2.9], dtype=F64)
    e, ws = P.choose(z, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}, "scale": 2.0})
    assert e == [0, 5, 4] and math.isclose(float(ws.sum()), 2.0) and math.isclose(float(ws[0] / ws[1]), math.exp(0.1))
    assert P.choose(z, {"experts": 6, "top": 3, "scale": 1.0})[0] == [0, 5, 2]
    assert math.isclose(float(P.tanh_norm(torch.tensor(2.0, dtype=F64), 0.5, 3.0, 0.25)), 3.0 * math.tanh(1.0) + 0.25)


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_plain_forward_is_causal_and_uses_every_tensor(name):
    cfg = CONFIGS[name]
    W = {k: v.to(F64) for k, v in random_weights(cfg, 3).items()}
    toks = tokens(cfg, 34, 1)
    raw = cfg.to_json()
    full = P.forward(raw, W, toks)
    assert torch.allclose(full[:21], P.forward(raw, W, toks[:21]))             # later tokens change nothing earlier
    for n in W:
        W2 = dict(W)
        W2[n] = W[n] + 0.3 * torch.arange(1, W[n].numel() + 1, dtype=F64).cos().reshape(W[n].shape)
        if ".mlp.e" in n and not any(x in n for x in (".e0.", ".e3.")):
            continue                                                           # (a few experts stand for all)
        assert not torch.allclose(full, P.forward(raw, W2, toks)), n


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cut_on_the_stand_in(name):
    cfg = CONFIGS[name]
    W = random_weights(cfg, 3)
    model = Model.from_tensors(cfg, W, dtype="float32", device="cpu", ops=CpuOps("float32"))
    reqs = {f"{name}{i}": tokens(cfg, n, i) for i, n in enumerate([37, 66, 5, 1, 18])}
    want = {rid: P.forward(cfg.to_json(), W, t).numpy() for rid, t in reqs.items()}
    for steps, pool in ((R.whole(reqs), 128), (R.tail_one_by_one(reqs, 9), 128), (R.portions(reqs, sizes=(3, 2, 11, 1)), 128),
                        (R.portions(reqs, sizes=(2,)), 128), (R.mixed(reqs, 192, seed=5), 192)):
        got = R.collect(steps, R.run_in_process(model, steps, pool), cfg.vocab)
        for rid in reqs:
            err = np.abs(got[rid] - want[rid]).max() / np.abs(want[rid]).max()
            assert err < 2e-4, (rid, err)


def test_greedy_generation_through_the_engine_on_the_stand_in():
    from bitwise_b200 import Engine, EngineConfig, SamplingParams
    cfg = CONFIGS["a"]
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
    assert tuple(tensors["l1.norm1.alpha"].shape) == ()
    toks = tokens(cfg, 30, 2)
    got = Model.load(folder, "float32", device="cpu", ops=CpuOps("float32")).logits(toks)
    want = P.forward(stored, tensors, toks).numpy()
    assert np.abs(got - want).max() < 2e-4 * np.abs(want).max()
