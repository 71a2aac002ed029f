"""Sazisun on the device against the plain implementation (tests/plain_sazisun.py).

Each new mechanism alone (the state-space recurrence with its state, in one walk and in portions, bit for bit the same; what
prepares and what finishes it; the norm without statistics; two maps over the same values with their difference, norm and gate;
the rotation of pairs with rescaled wavelengths on its way into the pages; softmax routing in groups; ungated experts' products
and the combination with a gated shared one), then whole models of several shapes in both precisions, the same requests cut in
every way (whole, token by token, portions down to two tokens, mixed batches over a pool whose pages and slots are used again),
a far token that one map looks for in a prompt and in decoding, long decoding, and greedy generation through the engine and its
scheduler and through the command line.
"""
import json
import math

import numpy as np
import pytest
import torch

import plain_sazisun as P
import replay_patterns as R
from sazisun_configs import CONFIGS, D, L, attention, random_weights, tokens
from test_zuzupel_gpu import DEV, SEQ, Batch, act, assess, close, d64, ops_of, row_errors, scattered_table, to_bf16
from bitwise_b200.config.sazisun import SazisunConfig

pytestmark = pytest.mark.gpu

F64 = torch.float64
DTYPES = ["float32", "bfloat16"]
WEIGHT_SEED = 3
_models, _plain = {}, {}


# ---- the recurrence ------------------------------------------------------------------------
# (heads, groups, state, value size): every layout of lanes and columns, sizes that are no multiple of 4
SHAPES = [(1, 1, 7, 5), (4, 2, 16, 16), (3, 3, 30, 9), (6, 2, 24, 32), (2, 1, 64, 48), (3, 1, 65, 3), (8, 2, 128, 64), (1, 1, 140, 8), (2, 1, 256, 12),
          (1, 1, 300, 6)]


class Walk:
    """The inputs of one sequence on the device as columns of wide rows, and the plain result."""

    def __init__(self, shape, n, g, far=None):
        self.H, self.G, self.N, self.vd = shape
        self.n = n
        r = lambda *s: torch.randn(*s, generator=g)
        self.x, self.B, self.C = r(n, self.H, self.vd), r(n, self.G, self.N) / math.sqrt(self.N), r(n, self.G, self.N)
        self.dt, self.rate, self.D = torch.rand(n, self.H, generator=g), 0.1 + torch.rand(self.H, generator=g), r(self.H)
        if far is not None:                       # nothing decays, and the last token asks for what token `far` wrote
            self.rate = torch.zeros(self.H)
            self.B[far] *= 40.0
            self.C[-1] = self.B[far]

    def plain(self):
        f = lambda t: t.to(F64)
        rep = self.H // self.G
        return P.space_scan(f(self.x), f(self.B).repeat_interleave(rep, 1), f(self.C).repeat_interleave(rep, 1), f(self.dt), f(self.rate), f(self.D))[0]


def run_walks(ops, walks, portions, state, slots):
    """Every step of ``portions`` is a list of (walk, first row, rows); one launch per step.  Returns the outputs by walk."""
    w0 = walks[0]
    H, G, N, vd = w0.H, w0.G, w0.N, w0.vd
    outs = {id(w): torch.zeros(w.n, H, vd, dtype=F64) for w in walks}
    for step in portions:
        b = Batch([(a, c) for _, a, c in step], [slots[id(w)] for w, _, _ in step])
        cat = lambda get: torch.cat([get(w)[a:a + c].reshape(c, -1) for w, a, c in step]).float()
        decay = lambda w: torch.exp(-w.rate.to(F64) * w.dt.to(F64))
        wide = torch.cat([cat(lambda w: w.x), cat(lambda w: w.B), cat(lambda w: w.C), cat(lambda w: w.dt), cat(decay)], 1).contiguous().to(DEV)
        x, B, C, dt, dec = wide.split([H * vd, G * N, G * N, H, H], 1)
        o = torch.full((b.n, H * vd), float("nan"), device=DEV)
        ops.state_scan("space", C, B, x, state, o, b, b.query_tiles(SEQ), H, N, vd, step=dt, decay=dec, skip=w0.D.to(DEV))
        r = 0
        for w, a, c in step:
            outs[id(w)][a:a + c] = d64(o)[r:r + c].view(c, H, vd)
            r += c
    return [outs[id(w)] for w in walks]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_recurrence_whole_and_in_portions(dtype, shape):
    """Three sequences, each in one walk, in portions of several sizes (down to two and one), and together with the others in
    one step: against the plain walk, and bit for bit the same in every cut.  Slots come dirty and out of order."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(sum(shape))
    first = Walk(shape, 83, g)
    walks = [first, Walk(shape, 40, g), Walk(shape, 9, g)]
    for w in walks[1:]:                                        # (weights of the layer, not of a sequence)
        w.rate, w.D = first.rate, first.D
    want = [w.plain() for w in walks]
    slots = {id(w): s for w, s in zip(walks, (3, 0, 4))}
    fresh = lambda: torch.randn(6, *ops.scan_state_shape("space", shape[0], shape[2], shape[3]), generator=torch.Generator().manual_seed(1)).to(DEV) * 7.0
    state = fresh()
    whole = run_walks(ops, walks, [[(w, 0, w.n)] for w in walks], state, slots)
    for got, w in zip(whole, want):
        close(got, w, "float32", f"{shape}", factor=2.0)
    assert torch.equal(state[[1, 2, 5]], fresh()[[1, 2, 5]])
    cuts = {"two at a time": [[(w, a, min(2, w.n - a))] for w in walks for a in range(0, w.n, 2)],
            "unequal": [[(first, 0, 33), (walks[1], 0, 1)], [(walks[1], 1, 38), (first, 33, 1), (walks[2], 0, 4)], [(first, 34, 32)],
                        [(walks[2], 4, 5), (walks[1], 39, 1), (first, 66, 17)]],
            "one by one together": [[(w, a, 1) for w in walks if a < w.n] for a in range(83)]}
    end = state
    for what, portions in cuts.items():
        st = fresh()
        for got, ref in zip(run_walks(ops, walks, portions, st, slots), whole):
            assert torch.equal(got, ref), f"{shape}, {what}: not the bits of the whole walk"
        assert torch.equal(st, end), f"{shape}, {what}: another state"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(4, 2, 16, 16), (2, 1, 64, 48), (2, 2, 128, 20)], ids=str)
def test_a_far_token_is_remembered(dtype, shape):
    ops = ops_of(dtype)
    w = Walk(shape, 500, torch.Generator().manual_seed(9), far=3)
    want = w.plain()
    without = Walk(shape, 500, torch.Generator().manual_seed(9), far=3)
    without.x = without.x.clone()
    without.x[3] = 0.0
    gap = float((want[-1] - without.plain()[-1]).abs().max())
    assert gap > 0.3 * float(want[-1].abs().max()), "the far token did not decide"
    for portions in ([[(w, 0, 500)]], [[(w, 0, 2)], [(w, 2, 3)], [(w, 5, 490)]] + [[(w, a, 1)] for a in range(495, 500)]):
        state = torch.full((1, *ops.scan_state_shape("space", w.H, w.N, w.vd)), 3.0, device=DEV)
        got = run_walks(ops, [w], portions, state, {id(w): 0})[0]
        assert float((got[-1] - want[-1]).abs().max()) < 1e-4 * gap


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,groups,state,vdim,taps", [(1, 1, 7, 5, 1), (4, 2, 16, 24, 4), (3, 3, 30, 9, 2), (6, 2, 128, 64, 3), (2, 1, 300, 132, 6), (40, 4, 8, 4, 5)])
def test_what_the_recurrence_reads(dtype, heads, groups, state, vdim, taps):
    """Convolution with a bias over portions of sequences, SiLU, steps and decays; the convolution's state, kept by the kernel
    itself (steps of one row per sequence) and by the update after it; short steps and steps of many rows."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(state + taps)
    r = lambda *s: torch.randn(*s, generator=g)
    inner = heads * vdim
    ch = inner + 2 * groups * state
    total = {0: 150, 1: 76, 2: 1}
    full, zlog = {s: r(n, ch) for s, n in total.items()}, {s: r(n, heads) * 3.0 for s, n in total.items()}
    conv, cb, bias, rate = r(ch, taps) * 0.6, r(ch) * 0.3, r(heads), r(heads).exp()
    want = {}
    for s in total:
        y = P.silu(P.causal_conv(full[s].to(F64), conv.to(F64), cb.to(F64)))
        t = P.step_sizes(zlog[s].to(F64), bias.to(F64))
        want[s] = torch.cat([y, t, torch.exp(-rate.to(F64) * t)], 1)
    st = torch.randn(5, max(taps - 1, 1), ch, generator=g).to(DEV) if taps > 1 else None
    slot, at = {0: 4, 1: 0, 2: 2}, {s: 0 for s in total}
    pad = -(2 * inner + 2 * groups * state + heads) % 8
    col = ch + (-ch) % 8
    for step in ([(0, 2), (1, 1)], [(0, 1), (1, 1), (2, 1)], [(0, 1)], [(0, 7), (1, 4)], [(0, 1)], [(0, 90), (1, 70)], [(0, 48)]):
        b = Batch([(at[s], c) for s, c in step], [slot[s] for s, _ in step])
        rows = lambda t: torch.cat([t[s][at[s]:at[s] + c] for s, c in step])
        u = torch.cat([torch.full((b.n, inner), 9.0), rows(full), rows(zlog), torch.full((b.n, pad), 9.0)], 1).contiguous().to(DEV)
        ready = torch.zeros(b.n, col + 2 * heads + (-2 * heads) % 4, device=DEV)
        keep = all(c == 1 for _, c in step)
        ops.space_prepare(u, inner, inner + ch, conv.t().contiguous().to(DEV), cb.to(DEV), st, bias.to(DEV), rate.to(DEV), ready, col, b, keep=keep)
        if st is not None and not keep:
            ops.conv_state_update(u[:, inner:inner + ch], st, b, taps, b.query_tiles(SEQ))
        ref = torch.cat([want[s][at[s]:at[s] + c] for s, c in step])
        close(ready[:, :ch], ref[:, :ch], "float32", "x, B, C")
        close(ready[:, col:col + heads], ref[:, ch:ch + heads], "float32", "steps")
        close(ready[:, col + heads:col + 2 * heads], ref[:, ch + heads:], "float32", "decays")
        for s, c in step:
            at[s] += c
            for j in range(taps - 1):
                p = at[s] - (taps - 1) + j
                assert torch.equal(st[slot[s], j].cpu(), full[s][p] if p >= 0 else torch.zeros(ch)), (s, at[s], j)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,groups", [(45, 3), (45, 1), (96, 2), (2048, 1), (4096, 8), (20, 5)])
def test_gated_norm_in_groups(dtype, width, groups):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width)
    n = 7
    o = torch.randn(n, width, generator=g).to(DEV) * torch.logspace(-2, 2, width).to(DEV)     # parts of unlike size
    wide = torch.randn(n, width + 8, generator=g).to(DEV) * 2.0
    w = (1.0 + 0.2 * torch.randn(width, generator=g)).to(DEV)
    for first in (0, 3):
        gate = wide[:, first:first + width]
        out = torch.zeros(n, width, dtype=act(dtype), device=DEV)
        ops.gated_group_norm(o, gate, w, 1e-3, out, groups)
        close(out, P.gated_group_norm(d64(o), d64(gate), d64(w), groups, 1e-3), dtype, "gated norm")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [50, 256, 1100, 4096])
def test_norm_without_statistics(dtype, width):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g).to(DEV)
    x, w, b, alpha = r(9, width) * 3.0, 1.0 + 0.2 * r(width), r(width), torch.tensor([0.37], device=DEV)
    x[0] *= 1e-3                                                   # where tanh is its argument
    x[1] *= 1e3                                                    # and where it is one
    ref = P.tanh_norm(d64(x), 0.37, d64(w), d64(b))
    out = torch.zeros(9, width, dtype=act(dtype), device=DEV)
    ops.tanh_norm(x, alpha, w, b, out)
    close(out, ref, dtype, "rows")
    rows = torch.tensor([8, 0, 3], dtype=torch.int32, device=DEV)
    ops.tanh_norm(x, alpha, w, b, out[:3], rows)
    close(out[:3], ref[[8, 0, 3]], dtype, "gathered rows")
    d, y = r(9, width), x.clone()
    ops.tanh_norm(y, alpha, w, b, out, d=d)
    assert torch.equal(y, x + d)
    close(out, P.tanh_norm(d64(x) + d64(d), 0.37, d64(w), d64(b)), dtype, "after a residual sum")


# ---- two maps ---------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims", [(4, 2, 16, 32, 8), (3, 3, 10, 6, 4), (6, 1, 64, 128, 64), (2, 2, 200, 24, 130), (2, 1, 36, 12, 2)])
def test_rotation_of_pairs_on_the_way_into_the_pages(dtype, heads, kv_heads, dim, vdim, dims):
    from bitwise_b200.parts.rope import PairRotaryEncoding, WavelengthScaling
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(dim)
    b = Batch([(0, 5), (37, 4), (250, 1), (15, 20)])
    page = 16
    table = scattered_table(b.seqs, page, g)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100}}
    cos, sin = PairRotaryEncoding(dims, 300.0, WavelengthScaling(4.0, 1.0, 4.0, 100), positions=300).rotary_tables(DEV)
    qc, kc_, vc_ = 2 * heads * dim, 2 * kv_heads * dim, kv_heads * vdim
    u = torch.randn(b.n, qc + kc_ + vc_ + 8, generator=g).to(DEV)[:, :qc + kc_ + vc_]
    pages = int(table.max()) + 1
    kc = torch.zeros(pages, 2 * kv_heads, page, dim, dtype=act(dtype), device=DEV)
    vc = torch.zeros(pages, kv_heads, page, vdim, dtype=act(dtype), device=DEV)
    q = torch.zeros(b.n, qc, dtype=act(dtype), device=DEV)
    ops.qkv_prepare(u, None, None, None, None, 1e-5, cos, sin, b, table, kc, vc, q, 2 * heads, 2 * kv_heads, dim, vdim, v_heads=kv_heads)
    turned = lambda t: P.rotate_pairs(t.reshape(b.n, -1, dim), b.positions, rot)
    close(q, turned(d64(u)[:, :qc]).reshape(b.n, -1), dtype, "queries")
    rows = lambda c: torch.stack([c[int(table[int(b.row_seq[r]), p // page]), :, p % page] for r, p in enumerate(b.positions)])
    close(rows(kc), turned(d64(u)[:, qc:qc + kc_]), dtype, "stored keys")
    close(rows(vc), d64(u)[:, qc + kc_:].reshape(b.n, kv_heads, vdim), dtype, "stored values")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 32, 16), (3, 3, 10, 6), (8, 1, 64, 128), (2, 2, 72, 144), (24, 2, 16, 64), (40, 1, 16, 32), (1, 1, 128, 256)])
@pytest.mark.parametrize("cap,plain", [(0.0, False), (7.0, False), (7.0, True)])
def test_a_far_key_of_one_map(dtype, heads, kv_heads, dim, vdim, cap, plain):
    """Keys at page, key-tile and span edges carry nearly all the weight of one of the two maps and none of the other's: rows of
    prompts' portions and single rows, contexts below and beyond a span; pages that nobody holds are rubbish."""
    ops = ops_of(dtype)
    if plain and dtype == "float32":
        pytest.skip("one kernel only")
    g = torch.Generator().manual_seed(heads * dim)
    page, T, scale, lam, keep, eps = 16, 720, 0.5, 0.62, 0.4, 1e-4
    table = scattered_table([(0, T), (0, T)], page, g)
    pages = int(table.max()) + 1
    kc = torch.full((pages, 2 * kv_heads, page, dim), 1e4, dtype=act(dtype), device=DEV)
    vc = torch.full((pages, kv_heads, page, vdim), 1e4, dtype=act(dtype), device=DEV)
    keys, vals = torch.randn(2, T, 2 * kv_heads, dim, generator=g) * 0.3, torch.randn(2, T, kv_heads, vdim, generator=g)
    direction = torch.randn(2, dim, generator=g)
    direction /= direction.norm(dim=-1, keepdim=True)
    edges = [0, 15, 16, 31, 32, 63, 64, 255, 256, 257, 511, 512, 700]
    for i, p in enumerate(edges):                       # the map that sees the key at an edge, by turns
        keys[:, p, i % 2::2] = direction[i % 2] * (5.0 + 0.4 * (p % 7))
    idx = torch.arange(T)
    for s in range(2):
        kc[table[s].long()[idx // page], :, idx % page] = keys[s].to(act(dtype)).to(DEV)
        vc[table[s].long()[idx // page], :, idx % page] = vals[s].to(act(dtype)).to(DEV)
    k64 = [kc[table[s].long()[idx // page], :, idx % page].to(F64).cpu() for s in range(2)]
    v64 = [vc[table[s].long()[idx // page], :, idx % page].to(F64).cpu() for s in range(2)]
    ops.plain_mixers(plain)
    try:
        for seqs in ([(690, 20), (3, 5)], [(512, 1), (255, 1)], [(256, 1), (16, 1)], [(0, 90), (256, 3)], [(500, 130), (31, 2)], [(0, 1), (15, 2)]):
            b = Batch(seqs)
            q = torch.randn(b.n, heads, 2, dim, generator=g) * 0.2 + direction * 3.0
            qd = q.reshape(b.n, -1).to(act(dtype)).to(DEV)
            wide = torch.randn(b.n, heads * vdim + 4, generator=g).to(DEV)
            for gate, group in ((wide[:, :heads * vdim], 1), (wide[:, 2:2 + heads], vdim), (None, 1)):
                out = torch.zeros(b.n, heads * vdim, dtype=act(dtype), device=DEV)
                ops.scored_attention(qd, kc, vc, table, out, 2 * heads, 2 * kv_heads, dim, vdim, scale, cap, False, None, 0, b,
                                     difference=(torch.tensor([lam], device=DEV), keep, eps, gate, group))
                q64 = d64(qd).view(b.n, heads, 2, dim)
                want = []
                for r, p in enumerate(b.positions):
                    s = int(b.row_seq[r])
                    kk = k64[s][:p + 1].view(p + 1, kv_heads, 2, dim).repeat_interleave(heads // kv_heads, 1)
                    vv = v64[s][:p + 1].repeat_interleave(heads // kv_heads, 1)
                    sc = torch.einsum("hmd,khmd->hmk", q64[r], kk) * scale
                    if cap:
                        sc = cap * torch.tanh(sc / cap)
                    a = torch.einsum("hmk,khd->hmd", torch.softmax(sc, -1), vv)
                    want.append(P.unit_rms(a[:, 0] - lam * a[:, 1], eps).reshape(-1) * keep)
                want = torch.stack(want)
                if gate is not None:
                    want = want * torch.sigmoid(d64(gate)).repeat_interleave(group, 1)
                close(out, want, dtype, f"rows {seqs}, gate of {group}", factor=2.0)
    finally:
        ops.plain_mixers(False)


# ---- routing and experts ---------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,groups,keep,top", [(8, 4, 2, 3), (5, 1, 1, 5), (64, 8, 3, 6), (7, 7, 2, 2), (160, 8, 2, 8), (6, 3, 3, 1)])
@pytest.mark.parametrize("rows", [1, 8, 33])
def test_softmax_routing_in_groups(dtype, experts, groups, keep, top, rows):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(experts + rows)
    wide = torch.randn(rows, experts + 3, generator=g) * 3.0
    wide[0, :experts] -= 200.0 * torch.rand(experts, generator=g)  # scores that underflow keep their order
    wide = wide.to(DEV)
    chosen = torch.zeros(rows, top, dtype=torch.int32, device=DEV)
    weights = torch.zeros(rows, top, device=DEV)
    ops.route(wide[:, :experts], None, groups, keep, top, 1.75, chosen, weights, scoring="softmax", group_max=True, sum_eps=1e-20)
    for r in range(rows):
        e, w = P.choose(d64(wide)[r, :experts], {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.75})
        assert chosen[r].tolist() == e, r
        assert float((d64(weights)[r] - w).abs().max()) < 1e-5, r
    # a group as the sum of its two largest, weights as they are: the other options with the same scores
    if experts // groups > 1:
        ops.route(wide[:, :experts], None, groups, keep, top, 0.5, chosen, weights, scoring="softmax")
        for r in range(1, rows):
            s = torch.softmax(d64(wide)[r, :experts], -1)
            two = s.view(groups, -1).topk(2, -1).values.sum(-1)
            best = two.topk(keep).indices
            allowed = torch.full((experts,), -1.0, dtype=F64)
            for j in best.tolist():
                per = experts // groups
                allowed[j * per:(j + 1) * per] = s[j * per:(j + 1) * per]
            v, i = allowed.topk(top)
            assert chosen[r].tolist() == i.tolist() and float((d64(weights)[r] - 0.5 * v).abs().max()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,experts,top,width,inner,shared", [(1, 5, 2, 50, 9, 13), (8, 8, 3, 64, 48, 32), (70, 6, 2, 96, 64, 80), (600, 4, 2, 128, 192, 64)])
def test_experts_with_the_square_of_relu_and_a_gated_shared_one(dtype, rows, experts, top, width, inner, shared):
    """The whole feed-forward part on its kernels (few rows, many, and lists long enough for the tcgen05 product)."""
    from bitwise_b200.parts import DenseFFN, RoutedFFN
    from bitwise_b200.parts.base import StepContext, Workspace
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width + rows)
    r = lambda *s: torch.randn(*s, generator=g)
    part = RoutedFFN(width, experts, top, inner, 0.0, 0.0, 1.3, 1, 1, correction=False, shared=DenseFFN(width, shared), scoring="softmax",
                     activation="relu2", group_score="max", sum_eps=1e-20, shared_gate="shared.sg")
    W = {s.name: (r(*s.shape) / math.sqrt(s.shape[1])).to(torch.bfloat16) for s in part.param_specs("m")}
    h = r(rows, width).to(torch.bfloat16)
    # the choice must not hang on rounding: one channel per expert with separated levels
    h[:, :experts] = torch.stack([torch.linspace(-1.5, 1.5, experts)[torch.randperm(experts, generator=g)] for _ in range(rows)]).to(torch.bfloat16)
    W["m.router"] = torch.zeros(experts, width, dtype=torch.bfloat16)
    W["m.router"][torch.arange(experts), torch.arange(experts)] = 2.0
    part.load_params({k: v.to(act(dtype)).to(DEV) for k, v in W.items()}, "m")
    zero = torch.zeros(1, dtype=torch.int32, device=DEV)
    ctx = StepContext(ops, Workspace(DEV, max(rows, 8)), rows, 1, zero, zero, zero, zero, zero, zero, zero, 0, rows)
    x0 = r(rows, width).to(DEV)
    x = x0.clone()
    part.forward(ctx, h.to(act(dtype)).to(DEV), x)
    cfg = {"router": {"experts": experts, "top": top, "scale": 1.3}, "shared": {"ff": shared}}
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = P.routed_ff(h.to(F64), W64, "m.", cfg)
    with P.rounding(to_bf16):
        slack = float((P.routed_ff(h.to(F64), W64, "m.", cfg) - want).abs().max())
    err = float((d64(x) - d64(x0) - want).abs().max())
    assert err <= (1e-5 * float(want.abs().max()) if dtype == "float32" else 2.0 * slack + 1e-4), (err, slack)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,groups,keep,top", [(8, 4, 2, 3), (5, 1, 1, 5), (64, 8, 3, 6), (256, 8, 4, 8)])
@pytest.mark.parametrize("rows", [1, 8, 16, 17])
def test_routing_and_its_lists_in_one_kernel(dtype, experts, groups, keep, top, rows):
    ops = ops_of(dtype)
    z = torch.randn(rows, experts, generator=torch.Generator().manual_seed(experts + rows)).to(DEV)
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device=DEV)
    out = []
    for together in (False, True):
        chosen, weights = i32(rows, top), torch.zeros(rows, top, device=DEV)
        lists = (i32(experts + 1), i32(2, experts + 1), i32(rows, top), i32(rows, top))
        options = dict(scoring="softmax", group_max=True, sum_eps=1e-20)
        if together:
            ops.route(z, None, groups, keep, top, 1.5, chosen, weights, lists=lists, **options)
        else:
            ops.route(z, None, groups, keep, top, 1.5, chosen, weights, **options)
            ops.group_rows(chosen, experts, *lists)
        out.append((chosen, weights, *lists))
    assert all(torch.equal(a, b) for a, b in zip(*out))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,width,inner", [(1, 64, 128), (8, 1024, 2048), (9, 80, 192), (16, 256, 64), (17, 256, 64), (5, 50, 36), (300, 128, 64)])
def test_a_product_and_the_norm_behind_it_in_one_kernel(dtype, rows, width, inner):
    """The bits of the product with its residual sum and of the stand-alone norm, in steps of few rows (one kernel on the
    serving precision) and of many; the same behind the experts' combination."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width + rows)
    r = lambda *s: torch.randn(*s, generator=g)
    x, w = r(rows, inner).to(act(dtype)).to(DEV), (r(width, inner) / math.sqrt(inner)).to(act(dtype)).to(DEV)
    res, nw, nb, alpha = r(rows, width).to(DEV), 1.0 + 0.2 * r(width).to(DEV), r(width).to(DEV), torch.tensor([0.7], device=DEV)
    norm = lambda: torch.zeros(rows, width, dtype=act(dtype), device=DEV)
    y, n1, y2, n2 = res.clone(), norm(), res.clone(), norm()
    ops.linear(x, w, y, residual=y)
    ops.tanh_norm(y, alpha, nw, nb, n1)
    before = ops.launches
    ops.linear(x, w, y2, residual=y2, then=(alpha, nw, nb, n2))
    if dtype == "bfloat16" and rows <= 16 and inner % 64 == 0:
        assert ops.launches - before == 1
    assert torch.equal(y, y2) and torch.equal(n1, n2)
    top = 2
    yy, wt, d, gate = r(rows * top, width).to(DEV), r(rows, top).to(DEV), r(rows, width).to(DEV), r(rows, 5).to(DEV)[:, 3:4]
    place = torch.randperm(rows * top, generator=g).to(torch.int32).reshape(rows, top).to(DEV)
    a, n1, b, n2 = res.clone(), norm(), res.clone(), norm()
    ops.combine(a, d, yy, place, wt, top, d_gate=gate)
    ops.tanh_norm(a, alpha, nw, nb, n1)
    ops.combine(b, d, yy, place, wt, top, d_gate=gate, then=(alpha, nw, nb, n2))
    assert torch.equal(a, b) and torch.equal(n1, n2)
    want = d64(res) + torch.sigmoid(d64(gate)) * d64(d) + (d64(wt)[:, :, None] * d64(yy)[place.cpu().long().reshape(-1)].view(rows, top, width)).sum(1)
    close(a, want, "float32", "combination")


# ---- whole models -------------------------------------------------------------------------------
def model_of(name, dtype):
    from bitwise_b200 import Model
    if (name, dtype) not in _models:
        _models[(name, dtype)] = Model.from_tensors(CONFIGS[name], random_weights(CONFIGS[name], WEIGHT_SEED), dtype=dtype, device=DEV)
    return _models[(name, dtype)]


def plain_pair(cfg, W, toks, collect=None):
    """The plain logits of one request, and the plain logits with everything rounded to bfloat16 that the serving
    precision stores in it: the second shows how large an error rounding alone causes for these weights."""
    exact = P.forward(cfg.to_json(), W, toks, collect).numpy()
    with P.rounding(to_bf16):
        rounded_ = P.forward(cfg.to_json(), W, toks).numpy()
    return exact, rounded_


def plain_logits(name, toks, rounded_too=False):
    key = (name, tuple(toks))
    if key not in _plain:
        _plain[key] = plain_pair(CONFIGS[name], random_weights(CONFIGS[name], WEIGHT_SEED), toks)
    return _plain[key] if rounded_too else _plain[key][0]


# lengths around the pages' (16) and the key tiles' and spans' edges (32, 256)
LENGTHS = {"a": [70, 41, 5, 300, 64, 17, 1, 131], "b": [100, 9, 290, 1, 65, 33], "c": [40, 270, 3, 17, 132], "d": [50, 33, 2, 100]}


def requests_of(name):
    return {f"{name}-{i}": tokens(CONFIGS[name], n, i) for i, n in enumerate(LENGTHS[name])}


def compare(name, dtype, got_by_request):
    errors, base = [], []
    for rid, toks in requests_of(name).items():
        want, rounded_ = plain_logits(name, toks, rounded_too=True)
        got = got_by_request[rid]
        assert got.shape == want.shape
        errors.append(row_errors(got, want))
        base.append(row_errors(rounded_, want))
    assess(errors, dtype, f"{name} {dtype} against the plain implementation", base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_and_layers(name, dtype):
    model = model_of(name, dtype)
    reqs = requests_of(name)
    steps = R.whole(reqs)
    compare(name, dtype, R.collect(steps, R.run_in_process(model, steps, 384), CONFIGS[name].vocab))
    if dtype == "float32":                                   # the stream after every layer, for one request
        from bitwise_b200.engine.replay import make_replay_stepper
        from bitwise_b200.engine.step import StepEntry
        toks = reqs[f"{name}-1"]
        want, caught = [], []
        P.forward(CONFIGS[name].to_json(), random_weights(CONFIGS[name], WEIGHT_SEED), toks, want)
        originals = [b.forward for b in model.decoder.blocks]
        try:
            for b, orig in zip(model.decoder.blocks, originals):
                b.forward = lambda ctx, x, cache, _o=orig, **k: (_o(ctx, x, cache, **k), caught.append(x.detach().clone()))
            make_replay_stepper(model, 384, use_graphs=False).run([StepEntry("r", toks, [])])
        finally:
            for b in model.decoder.blocks:
                del b.forward
        assert len(caught) == len(want)
        for i, (got, w) in enumerate(zip(caught, want)):
            close(got, w, "float32", f"stream after layer {i}", factor=4.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_every_cut_gives_the_same_logits(name, dtype):
    model = model_of(name, dtype)
    reqs = requests_of(name)
    vocab = CONFIGS[name].vocab
    whole = R.collect(R.whole(reqs), R.run_in_process(model, R.whole(reqs), 384), vocab)
    cuts = {"token by token": (R.tail_one_by_one(reqs, 40), 384), "portions": (R.portions(reqs), 384),
            "portions of two": (R.portions(reqs, sizes=(2,)), 384), "mixed": (R.mixed(reqs, 512, seed=7), 512),
            "mixed, a tight pool": (R.mixed(reqs, 400, seed=8, max_live=3), 400)}
    for what, (steps, pool) in cuts.items():
        got = R.collect(steps, R.run_in_process(model, steps, pool, max_live=4), vocab)
        compare(name, dtype, got)
        for rid in reqs:                                      # and against the whole prompt, beyond rounding nothing
            err = np.abs(got[rid] - whole[rid]).max() / np.abs(whole[rid]).max()
            assert err <= (1e-4 if dtype == "float32" else 0.05), (what, rid, err)


def marked_model(dtype, which):
    """Two attention layers, the second on the first one's keys, whose map ``which`` alone looks along the first channels: a
    token whose embedding is large along one of them is found by another such token, however far away."""
    from bitwise_b200 import Model
    cfg = SazisunConfig(vocab=40, width=32, eps=1e-5, layers=(
        L(attention(heads=2, kv_heads=1, dim=16, vdim=16, scale=4.0, diff=0.4, softcap=40.0, dims=0), D(24)),
        L(attention(heads=2, kv_heads=1, dim=16, vdim=16, scale=4.0, diff=0.2, softcap=40.0, dims=0, kv_from=0), None)))
    W = random_weights(cfg, 5)
    look, none = torch.zeros(16, 32), torch.zeros(16, 32)
    look[:, :16] = torch.eye(16)
    maps = [look, none] if which == 0 else [none, look]
    for i in range(2):
        W[f"l{i}.mix.q"] = torch.cat(maps * 2).to(torch.bfloat16)
        W[f"l{i}.mix.lq1"] = W[f"l{i}.mix.lk1"] = torch.full((16,), 0.25, dtype=torch.bfloat16)      # lambda = e - 1 + diff
        W[f"l{i}.mix.lq2"] = torch.zeros(16, dtype=torch.bfloat16)
    W["l0.mix.k"] = torch.cat([look, look]).to(torch.bfloat16)
    for n in ("l0.norm1", "l1.norm1"):
        W[n + ".b"], W[n], W[n + ".alpha"] = torch.zeros_like(W[n]), torch.ones_like(W[n]), torch.tensor(0.5, dtype=torch.bfloat16)
    W["embed"] *= 0.6
    W["embed"][:, 0] = 0.0
    W["embed"][38:, :16] = 0.0
    W["embed"][38:, 0] = 6.0
    return cfg, W, Model.from_tensors(cfg, W, dtype=dtype, device=DEV)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", [0, 1])
@pytest.mark.parametrize("at", [0, 15, 16, 31, 255, 256])
def test_a_far_marked_token_decides(dtype, which, at):
    cfg, W, model = marked_model(dtype, which)
    total = 330
    base = [t % 38 for t in tokens(cfg, total, 1)]
    base[-1] = 39
    without = P.forward(cfg.to_json(), W, base)[-1].numpy()
    toks = list(base)
    toks[at] = 38
    want, rounded_ = plain_pair(cfg, W, toks)
    gap = np.abs(want[-1] - without).max()
    assert gap > 0.05 * np.abs(without).max(), "the far token did not decide"
    for steps in (R.portions({"r": toks}, sizes=(61, 2, 90, 47)), R.tail_one_by_one({"r": toks}, tail=total - at - 1 if at > 250 else 20)):
        got = R.collect(steps, R.run_in_process(model, steps, 384), cfg.vocab)["r"]
        assess([row_errors(got, want)], dtype, f"marked token at {at}", [row_errors(rounded_, want)])
        assert np.abs(got[-1] - want[-1]).max() < 0.2 * gap


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_over_reused_pages(dtype):
    # one request decoded token by token from position 3 to past 500 (pages, key tiles and spans are crossed one
    # position at a time) while others come and go in the pool and in the slots
    name = "a"
    model = model_of(name, dtype)
    toks = tokens(CONFIGS[name], 520, 99)
    others = {f"o{i}": tokens(CONFIGS[name], n, 50 + i) for i, n in enumerate([30, 64, 100, 7, 65, 120])}
    from bitwise_b200.engine.replay import make_replay_stepper
    from bitwise_b200.engine.step import StepEntry
    stepper = make_replay_stepper(model, 576 + 128 + 64, max_live=3)
    queue = list(others.items())
    live = None
    errors, base = [], []
    want, want_rounded = plain_logits(name, toks, rounded_too=True)
    stepper.run([StepEntry("long", toks[:3], [2])])
    for p in range(3, len(toks)):
        entries = [StepEntry("long", toks[p:p + 1], [0])]
        if live is None and queue and p % 7 == 0:
            live = [queue.pop(0), 0]
        if live is not None:
            (rid, ot), at = live
            c = min(len(ot) - at, 1 + p % 9)
            entries.append(StepEntry(rid, ot[at:at + c], [c - 1]))
            live[1] += c
        out = stepper.run(entries).float().cpu().numpy()
        errors.append(row_errors(out[0], want[p]))
        base.append(row_errors(want_rounded[p], want[p]))
        if live is not None:
            w, wr = plain_logits(name, live[0][1], rounded_too=True)
            errors.append(row_errors(out[1], w[live[1] - 1]))
            base.append(row_errors(wr[live[1] - 1], w[live[1] - 1]))
            if live[1] == len(live[0][1]):
                stepper.finish(live[0][0])
                live = None
    assert not queue
    stepper.finish("long")
    assert stepper.manager.all_free()
    assess(errors, dtype, "long decoding", base)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["a", "d"])
def test_greedy_generation_through_the_engine(dtype, name):
    from bitwise_b200 import Engine, EngineConfig, SamplingParams
    model = model_of(name, dtype)
    cfg = CONFIGS[name]
    prompts = [tokens(cfg, n, 200 + i) for i, n in enumerate([5, 40, 17, 1, 33])]
    new = 12
    # a pool that does not hold all requests at once and a token budget below the longest prompt
    eng = Engine(model, EngineConfig(num_blocks=12, block_size=16, max_batched_tokens=24, max_num_seqs=3))
    got = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=new, ignore_eos=True))
    W = random_weights(cfg, WEIGHT_SEED)
    for prompt, out in zip(prompts, got):
        assert len(out) == new
        seq = list(prompt)
        for t in out:
            row = P.forward(cfg.to_json(), W, seq)[-1].numpy()
            if dtype == "float32":
                assert t == int(row.argmax()) or row.max() - row[t] < 1e-4 * np.abs(row).max()
            else:
                assert row.max() - row[t] <= 0.05 * np.abs(row).max(), "the chosen token is no near-maximum"
            seq.append(t)
    assert eng.manager.all_free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_requests_decode_in_filled_up_steps(dtype):
    """More than eight requests decode together: on the serving precision such steps are filled up with rows of no request
    and replayed as graphs.  Each request's tokens must be those it yields alone."""
    from bitwise_b200 import Engine, EngineConfig, SamplingParams
    model = model_of("a", dtype)
    cfg = CONFIGS["a"]
    prompts = [tokens(cfg, 3 + (5 * i) % 37, 700 + i) for i in range(11)]
    sp = SamplingParams(temperature=0.0, max_new_tokens=20, ignore_eos=True)
    eng = Engine(model, EngineConfig(num_blocks=80, block_size=16, max_batched_tokens=128, max_num_seqs=11))
    together = eng.generate(prompts, sp)
    for i in (0, 3, 10):
        alone = Engine(model, EngineConfig(num_blocks=80, block_size=16, max_batched_tokens=128, max_num_seqs=1)).generate([prompts[i]], sp)
        assert together[i] == alone[0], i


@pytest.mark.parametrize("dtype", DTYPES)
def test_simulated_traces_reproduce_requests_run_alone(dtype):
    # the engine's simulator: random requests, budgets and pools, preemption with recomputation; a request's tokens
    # and the fingerprint of its logits must be those it yields alone on an idle engine
    from bitwise_b200.engine.simulate import run_traces
    out = run_traces(model_of("a", dtype), traces=8, seed=5)
    assert out.traces == 8 and out.requests_checked > 10
    assert out.violations == 0, (out.token_mismatch, out.fingerprint_mismatch, out.hangs, out.leaks)


def test_command_line_random_folder_replay_and_generation(tmp_path):
    """``bitwise_b200 random`` writes a Sazisun folder from a config.json; ``bin/trace_run`` replays a mixed schedule
    on it and ``bitwise_b200 generate`` decodes greedily: both as a user calls them, both against the plain
    implementation on the folder's own tensors."""
    import os
    import subprocess
    import sys
    from bitwise_b200.weights.safetensors_io import SafetensorsFile
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = CONFIGS["b"]
    (tmp_path / "config.json").write_text(json.dumps(cfg.to_json()))
    folder = tmp_path / "model"
    run = lambda *a, **k: subprocess.run([sys.executable, *a], capture_output=True, text=True, timeout=900, **k)
    p = run(os.path.join(root, "bin", "bitwise_b200"), "random", "--config", str(tmp_path / "config.json"), "--seed", "11",
            "--out", str(folder), "--dtype", "bfloat16", "--std", "0.2", "--norm-jitter", "0.2")
    assert p.returncode == 0, p.stderr[-2000:]
    f = SafetensorsFile(str(folder / "model.safetensors"))
    W = {n: f.tensor(n).clone() for n in f.names()}
    raw = json.load(open(folder / "config.json"))
    reqs = {f"q{i}": tokens(cfg, n, 300 + i) for i, n in enumerate([33, 70, 2, 19])}
    steps = R.mixed(reqs, 192, seed=8)
    out = tmp_path / "out"
    p = run(os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
            "--max-tokens", "192", input="".join(json.dumps(s) + "\n" for s in steps))
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.split("\n") if l.startswith("done")] == [f"done {s['step']}" for s in steps]
    outs = {s["step"]: np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(-1, cfg.vocab) for s in steps}
    got = R.collect(steps, outs, cfg.vocab)
    for rid, toks in reqs.items():
        want = P.forward(raw, W, toks).numpy()
        assert np.abs(got[rid] - want).max() <= 1e-4 * np.abs(want).max(), rid
    prompt = reqs["q3"]
    p = run(os.path.join(root, "bin", "bitwise_b200"), "generate", "--model", str(folder), "--dtype", "float32",
            "--max-new-tokens", "6", "--ignore-eos", "--temperature", "0", "--prompt-ids", ",".join(map(str, prompt)))
    assert p.returncode == 0, p.stderr[-2000:]
    seq = list(prompt)
    for t in json.loads(p.stdout.strip().split("\n")[0])["tokens"]:
        row = P.forward(raw, W, seq)[-1].numpy()
        assert t == int(row.argmax()) or row.max() - row[t] < 1e-4 * np.abs(row).max()
        seq.append(t)
