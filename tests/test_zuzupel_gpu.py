"""Zuzupel on the device against the plain implementation (tests/plain_zuzupel.py).

Each new mechanism alone (the three recurrences with their state, in one walk and in portions, bit for bit the same; what
prepares and what finishes them; the token shift; the half-layout rotation on its way into the pages; attention inside
chunks; the mean of two mixers and the norm behind it; activations in a product's epilogue), then whole models of several shapes
in both precisions, the same requests cut in every way (whole, token by token, portions down to two tokens, mixed batches over
a pool whose pages and slots are used again), a key just inside and just outside a chunk in a prompt and in decoding, memory of a
far token, long decoding, and greedy generation through the engine and its scheduler and through the command line.
"""
import json
import math

import numpy as np
import pytest
import torch

import plain_zuzupel as P
import replay_patterns as R
from zuzupel_configs import CONFIGS, L, pair, random_weights, tokens
from bitwise_b200.config.zuzupel import ZuzupelConfig

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}   # relative to the largest reference value
F64 = torch.float64
SEQ = 1 << 20                                  # one query tile per sequence
WEIGHT_SEED = 3
_models, _plain = {}, {}


def to_bf16(a):
    return a.to(torch.bfloat16).to(F64)


def ops_of(dtype):
    from bitwise_b200.kernels.ops import get_ops
    return get_ops(dtype)


def act(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def d64(t):
    return t.detach().to(F64).cpu()


def close(got, want, dtype, what="", factor=1.0):
    got = d64(got) if isinstance(got, torch.Tensor) else torch.as_tensor(got, dtype=F64)
    want = torch.as_tensor(want, dtype=F64)
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    err = float((got - want).abs().max() / max(float(want.abs().max()), 1e-30))
    assert err <= TOL[dtype] * factor, f"{what}: relative error {err:.3g}"


class Batch:
    """What the kernels read of a step: rows of sequences with their positions and slots, and query tiles."""

    def __init__(self, seqs, slots=None):
        # seqs: list of (first position, rows); one block-table row each
        pos, row_seq, seq_pos0, seq_row0 = [], [], [], []
        r = 0
        for s, (p0, cnt) in enumerate(seqs):
            seq_pos0.append(p0), seq_row0.append(r)
            pos += list(range(p0, p0 + cnt))
            row_seq += [s] * cnt
            r += cnt
        self.i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
        self.n, self.seqs, self.positions = r, seqs, pos
        self.pos, self.row_seq = self.i32(pos), self.i32(row_seq)
        self.seq_pos0, self.seq_row0 = self.i32(seq_pos0), self.i32(seq_row0 + [r])
        self.slots = list(slots) if slots is not None else list(range(len(seqs)))
        self.seq_slot = self.i32(self.slots)
        self.max_keys = max(pos) + 1

    def query_tiles(self, tile_rows):
        t_seq, t_row0, t_rows = [], [], []
        r = 0
        for s, (p0, cnt) in enumerate(self.seqs):
            for a in range(0, cnt, tile_rows):
                t_seq.append(s), t_row0.append(r + a), t_rows.append(min(tile_rows, cnt - a))
            r += cnt
        return self.i32(t_seq), self.i32(t_row0), self.i32(t_rows), len(t_seq)


def scattered_table(seqs, page, g, spare=5):
    """A block table [seqs, blocks] over a pool whose pages are handed out in no order."""
    blocks = (max(p0 + cnt for p0, cnt in seqs) + page - 1) // page
    perm = torch.randperm(len(seqs) * blocks + spare, generator=g)[:len(seqs) * blocks]
    return perm.to(torch.int32).reshape(len(seqs), blocks).to(DEV)


# ---- the recurrences -----------------------------------------------------------------------
# (heads, query/key heads, key size, value size): every layout of lanes and columns, sizes that are no multiple of 4
SHAPES = [(1, 1, 7, 5), (4, 2, 16, 16), (3, 3, 30, 9), (6, 2, 24, 32), (2, 1, 64, 48), (3, 1, 65, 3), (2, 2, 128, 20), (1, 1, 140, 8),
          (2, 1, 256, 12), (1, 1, 300, 6)]


class Walk:
    """The inputs of one sequence of a recurrence, on the device as columns of wide rows, and the plain result."""

    def __init__(self, mode, shape, n, g, far=None):
        H, G, dim, vd = shape
        if mode != "delta":
            G = H
        self.mode, self.H, self.G, self.dim, self.vd, self.n = mode, H, G, dim, vd, n
        r = lambda *s: torch.randn(*s, generator=g)
        q, k, v = r(n, G, dim) / math.sqrt(dim), r(n, G, dim), r(n, H, vd)
        self.extra = {}
        if mode == "delta":
            k = k / k.norm(dim=-1, keepdim=True)
            decay, beta = 0.9 + 0.1 * torch.rand(n, H, dim, generator=g), torch.rand(n, H, generator=g)
            if far is not None:
                # the value at token `far` is written at a key that no other token touches, and nothing decays
                decay, beta[far] = torch.ones_like(decay), 1.0
                k[:, :, 0] = 0.0
                k = k / k.norm(dim=-1, keepdim=True).clamp_min(1e-9)
                k[far], q[-1] = 0.0, 0.0
                k[far, :, 0], q[-1, :, 0] = 1.0, 1.0
            self.decay, self.beta = decay, beta
        elif mode == "bonus":
            self.z, self.z0, self.u = r(n, H, dim) - 2.0, 0.5 * r(H, dim), r(H, dim)
            if far is not None:
                self.z = self.z - 30.0                     # decays of one
                k[far] *= 40.0
                q[-1] = k[far]
        else:
            self.i, self.f, self.ib, self.fb, self.cap = 2.0 * r(n, H), r(n, H) + 3.0, r(H), r(H), 6.0
            if far is not None:
                self.cap, self.f = 30.0, r(n, H) + 28.0    # forget gates open
                self.i[far] = 25.0
                q[-1] = k[far] / k[far].norm(dim=-1, keepdim=True)
        self.q, self.k, self.v = q, k, v

    def plain(self):
        f = lambda t: t.to(F64)
        rep = self.H // self.G
        q, k = f(self.q).repeat_interleave(rep, 1), f(self.k).repeat_interleave(rep, 1)
        if self.mode == "delta":
            return P.delta_scan(q, k, f(self.v), f(self.decay), f(self.beta))[0]
        if self.mode == "bonus":
            return P.bonus_scan(q, k, f(self.v), torch.exp(-torch.exp(f(self.z) + f(self.z0))), f(self.u))[0]
        i = self.cap * torch.tanh((f(self.i) + f(self.ib)) / self.cap)
        fg = P.log_sigmoid(self.cap * torch.tanh((f(self.f) + f(self.fb)) / self.cap))
        return P.matrix_memory_scan(q, k, f(self.v), i, fg)[0]


def run_walks(ops, walks, portions, state, slots):
    """Every step of ``portions`` is a list of (walk, first row, rows); one launch per step.  Returns the outputs by
    walk, finished: divided by the normaliser for the matrix memory."""
    w0 = walks[0]
    mode, H, G, dim, vd = w0.mode, w0.H, w0.G, w0.dim, w0.vd
    outs = {id(w): torch.zeros(w.n, H, vd, dtype=F64) for w in walks}
    for step in portions:
        b = Batch([(a, c) for _, a, c in step], [slots[id(w)] for w, _, _ in step])
        cat = lambda get: torch.cat([get(w)[a:a + c].reshape(c, -1) for w, a, c in step]).float()
        # q | k | v as columns of one wide row where their offsets allow 16-byte reads or do not: both occur
        wide = torch.cat([cat(lambda w: w.q), cat(lambda w: w.k), cat(lambda w: w.v)], 1).contiguous().to(DEV)
        q, k, v = wide[:, :G * dim], wide[:, G * dim:2 * G * dim], wide[:, 2 * G * dim:]
        extra, aux = {}, None
        if mode == "delta":
            qk = torch.einsum("nhd,nhd->nh", cat(lambda w: w.q).view(-1, G, dim), cat(lambda w: w.k).view(-1, G, dim))
            bq = torch.cat([cat(lambda w: w.beta), qk], 1).contiguous().to(DEV)
            extra = dict(decay=cat(lambda w: w.decay).to(DEV), beta=bq[:, :H], qk=bq[:, H:])
        elif mode == "bonus":
            extra = dict(decay=cat(lambda w: w.z).to(DEV), decay_bias=w0.z0.reshape(-1).to(DEV), bonus=w0.u.reshape(-1).to(DEV))
        else:
            aux = torch.zeros(b.n, H * 2, device=DEV)
            gates = torch.cat([cat(lambda w: w.i), cat(lambda w: w.f)], 1).contiguous().to(DEV)
            extra = dict(inp=gates[:, :H], forget=gates[:, H:], inp_bias=w0.ib.to(DEV), forget_bias=w0.fb.to(DEV), cap=w0.cap, aux=aux)
        o = torch.full((b.n, H * vd), float("nan"), device=DEV)
        ops.state_scan(mode, q, k, v, state, o, b, b.query_tiles(SEQ), H, dim, vd, **extra)
        y = d64(o).view(b.n, H, vd)
        if aux is not None:
            a2 = d64(aux).view(b.n, H, 2)
            y = y / (torch.maximum(a2[..., 0].abs(), torch.exp(-a2[..., 1])) + 1e-6)[..., None]
        r = 0
        for w, a, c in step:
            outs[id(w)][a:a + c] = y[r:r + c]
            r += c
    return [outs[id(w)] for w in walks]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", ["delta", "bonus", "memory"])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_recurrence_whole_and_in_portions(dtype, mode, shape):
    """Three sequences, each in one walk, in portions of several sizes (down to two and one), and together with the others in
    one step: against the plain walk, and bit for bit the same in every cut.  Slots come dirty and out of order."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(sum(shape) + len(mode))
    first = Walk(mode, shape, 83, g)
    walks = [first, Walk(mode, shape, 40, g), Walk(mode, shape, 9, g)]
    for w in walks[1:]:                                        # (weights of the layer, not of a sequence)
        for n in ("z0", "u", "ib", "fb", "cap"):
            if hasattr(first, n):
                setattr(w, n, getattr(first, n))
    want = [w.plain() for w in walks]
    H, dim, vd = first.H, first.dim, first.vd
    slots = {id(w): s for w, s in zip(walks, (3, 0, 4))}
    fresh = lambda: torch.randn(6, *ops.scan_state_shape(mode, H, dim, vd), generator=torch.Generator().manual_seed(1)).to(DEV) * 7.0
    state = fresh()
    whole = run_walks(ops, walks, [[(w, 0, w.n)] for w in walks], state, slots)
    for got, w in zip(whole, want):
        close(got, w, "float32", f"{mode} {shape}", factor=5.0 if dtype == "float32" else 20.0)
    untouched = fresh()
    assert torch.equal(state[[1, 2, 5]], untouched[[1, 2, 5]])
    cuts = {"two at a time": [[(w, a, min(2, w.n - a))] for w in walks for a in range(0, w.n, 2)],
            "unequal": [[(first, 0, 33), (walks[1], 0, 1)], [(walks[1], 1, 38), (first, 33, 1), (walks[2], 0, 4)], [(first, 34, 32)],
                        [(walks[2], 4, 5), (walks[1], 39, 1), (first, 66, 17)]],
            "one by one together": [[(w, a, 1) for w in walks if a < w.n] for a in range(83)]}
    end = state
    for what, portions in cuts.items():
        st = fresh()
        for got, ref in zip(run_walks(ops, walks, portions, st, slots), whole):
            assert torch.equal(got, ref), f"{mode} {shape}, {what}: not the bits of the whole walk"
        assert torch.equal(st, end), f"{mode} {shape}, {what}: another state"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("mode", ["delta", "bonus", "memory"])
@pytest.mark.parametrize("shape", [(4, 2, 16, 16), (2, 1, 64, 48), (2, 2, 128, 20)], ids=str)
def test_a_far_token_is_remembered(dtype, mode, shape):
    """What token 3 wrote stands out in the state and is what the last of 500 tokens asks for."""
    ops = ops_of(dtype)
    w = Walk(mode, shape, 500, torch.Generator().manual_seed(9), far=3)
    want = w.plain()
    without = Walk(mode, shape, 500, torch.Generator().manual_seed(9), far=3)
    without.v = without.v.clone()
    without.v[3] = 0.0
    gap = float((want[-1] - without.plain()[-1]).abs().max())
    assert gap > 0.3 * float(want[-1].abs().max()), "the far token did not decide"
    for portions in ([[(w, 0, 500)]], [[(w, 0, 2)], [(w, 2, 3)], [(w, 5, 490)]] + [[(w, a, 1)] for a in range(495, 500)]):
        state = torch.full((1, *ops.scan_state_shape(mode, w.H, w.dim, w.vd)), 3.0, device=DEV)
        got = run_walks(ops, [w], portions, state, {id(w): 0})[0]
        assert float((got[-1] - want[-1]).abs().max()) < (1e-3 if dtype == "float32" else 1e-2) * gap + 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,vdim", [(1, 5), (3, 32), (6, 40), (2, 256), (5, 300)])
def test_scan_finish(dtype, heads, vdim):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(vdim)
    n = 7
    o = torch.randn(n, heads * vdim, generator=g).to(DEV)
    wide = torch.randn(n, heads * vdim + 5, generator=g).to(DEV) * 2.0
    gate = wide[:, 3:3 + heads * vdim]
    aux = torch.randn(n, heads * 2, generator=g).to(DEV) * 2.0
    out = torch.zeros(n, heads * vdim, dtype=act(dtype), device=DEV)
    for per_head in (False, True):
        w = (1.0 + 0.2 * torch.randn(heads * vdim if per_head else vdim, generator=g)).to(DEV)
        w64 = d64(w).reshape(-1, vdim)
        for kind in ("sigmoid", "silu"):
            z = d64(gate)
            act64 = torch.sigmoid(z) if kind == "sigmoid" else P.silu(z)
            ops.scan_finish(o, w, gate, 1e-3, out, heads, vdim, gate_kind=kind)
            y = d64(o).view(n, heads, vdim)
            close(out, (P.unit_rms(y, 1e-3) * w64).reshape(n, -1) * act64, dtype, f"finish {kind}")
        ops.scan_finish(o, w, gate, 1e-3, out, heads, vdim, aux=aux, q_scale=0.3)
        a = d64(aux).view(n, heads, 2)
        y = 0.3 * y / (torch.maximum((0.3 * a[..., 0]).abs(), torch.exp(-a[..., 1])) + 1e-6)[..., None]
        close(out, (P.unit_rms(y, 1e-3) * w64).reshape(n, -1) * torch.sigmoid(d64(gate)), dtype, "finish with a normaliser")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(1, 1, 7, 5, 1), (4, 2, 16, 24, 4), (3, 3, 30, 9, 2), (6, 2, 128, 64, 3), (2, 1, 300, 132, 5)])
def test_what_the_delta_rule_reads(dtype, heads, kv_heads, dim, vdim, taps):
    """Convolution over portions of sequences, SiLU, unit vectors, decays, beta, q . k; the convolution's state, kept by the
    kernel itself (steps of one row per sequence) and by the update after it."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(dim + taps)
    r = lambda *s: torch.randn(*s, generator=g)
    ch = 2 * kv_heads * dim + heads * vdim
    pad = -ch % 8
    total = {0: 23, 1: 6, 2: 1}
    full = {s: r(n, ch) for s, n in total.items()}
    blog = {s: r(n, heads) for s, n in total.items()}
    zlog = {s: r(n, heads * dim) * 2.0 for s, n in total.items()}
    conv, bias, alog = r(ch, taps) * 0.6, r(heads * dim), r(heads) * 0.5
    q_scale = dim ** -0.5
    want = {}
    for s in total:
        y = P.silu(P.causal_conv(full[s].to(F64), conv.to(F64)))
        q = P.unit_length(y[:, :kv_heads * dim].reshape(-1, kv_heads, dim)) * q_scale
        k = P.unit_length(y[:, kv_heads * dim:2 * kv_heads * dim].reshape(-1, kv_heads, dim))
        n = total[s]
        ready = torch.cat([q.reshape(n, -1), k.reshape(n, -1), y[:, 2 * kv_heads * dim:], torch.sigmoid(blog[s].to(F64)), (q * k).sum(-1)], 1)
        decay = torch.exp(-torch.exp(alog.to(F64))[None, :, None] * P.softplus((zlog[s] + bias).to(F64)).reshape(n, heads, dim))
        want[s] = (ready, decay.reshape(n, -1))
    state = torch.randn(5, max(taps - 1, 1), ch, generator=g).to(DEV) if taps > 1 else None
    slot = {0: 4, 1: 0, 2: 2}
    at = {s: 0 for s in total}
    for step in ([(0, 2), (1, 1)], [(0, 1), (1, 1), (2, 1)], [(0, 1)], [(0, 7), (1, 4)], [(0, 1)], [(0, 11)]):
        b = Batch([(at[s], c) for s, c in step], [slot[s] for s, _ in step])
        rows = lambda t: torch.cat([t[s][at[s]:at[s] + c] for s, c in step])
        u = torch.cat([rows(full), torch.zeros(b.n, pad), rows(blog)], 1).contiguous().to(DEV)
        z = torch.cat([rows(zlog), torch.ones(b.n, 3)], 1).contiguous().to(DEV)
        ready = torch.zeros(b.n, ch + heads + kv_heads + (-(ch + heads + kv_heads)) % 4, device=DEV)
        keep = all(c == 1 for _, c in step)
        ops.delta_prepare(u, ch + pad, conv.t().contiguous().to(DEV), state, z[:, :heads * dim], bias.to(DEV), alog.to(DEV), ready, b, heads,
                          kv_heads, dim, vdim, q_scale, keep=keep)
        if state is not None and not keep:
            ops.conv_state_update(u[:, :ch], state, b, taps, b.query_tiles(SEQ))
        close(ready[:, :ch + heads + kv_heads], torch.cat([want[s][0][at[s]:at[s] + c] for s, c in step]), "float32", "q, k, v, beta, q.k", 3.0)
        close(z[:, :heads * dim], torch.cat([want[s][1][at[s]:at[s] + c] for s, c in step]), "float32", "decays", 3.0)
        assert float((z[:, heads * dim:] - 1.0).abs().max()) == 0.0
        for s, c in step:
            at[s] += c
            for j in range(taps - 1):
                p = at[s] - (taps - 1) + j
                ref = full[s][p] if p >= 0 else torch.zeros(ch)
                assert torch.equal(state[slot[s], j].cpu(), ref), (s, at[s], j)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [50, 256, 1100])
def test_token_shift(dtype, width):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width)
    full = [torch.randn(n, width, generator=g) for n in (19, 5)]
    mu = torch.rand(5, width, generator=g)
    want = [torch.stack([x.to(F64) + (P.previous_rows(x.to(F64)) - x.to(F64)) * mu[s].to(F64) for s in range(5)]) for x in full]
    last = torch.randn(4, 1, width, generator=g).to(DEV)
    at, slot = [0, 0], [3, 1]
    for step in ([(0, 1)], [(0, 6), (1, 2)], [(0, 1), (1, 1)], [(1, 2), (0, 11)]):
        b = Batch([(at[s], c) for s, c in step], [slot[s] for s, _ in step])
        x = torch.cat([full[s][at[s]:at[s] + c] for s, c in step]).to(DEV)
        out = torch.zeros(5, b.n, width, dtype=act(dtype), device=DEV)
        keep = all(c == 1 for _, c in step)
        ops.shift_mix(x, mu.to(DEV), last, out, b, keep=keep)
        if not keep:
            ops.conv_state_update(x, last, b, 2, b.query_tiles(SEQ))
        close(out, torch.cat([want[s][:, at[s]:at[s] + c] for s, c in step], 1), dtype, "mixes")
        for s, c in step:
            at[s] += c
            assert torch.equal(last[slot[s], 0].cpu(), full[s][at[s] - 1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,rows", [(50, 7), (256, 33), (1500, 4), (8, 1)])
def test_norms_behind_a_sublayer(dtype, width, rows):
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)
    a, b, x0 = (r(rows, width) * 3.0 + 1.5).to(DEV), (r(rows, width) * 0.1).to(DEV), r(rows, width).to(DEV)
    w, wa, wb = ((1.0 + 0.2 * r(width)).to(DEV) for _ in range(3))
    rounded = torch.zeros(rows, width, dtype=act(dtype), device=DEV)
    # the summed row, rounded, instead of a next norm
    for op, plain in ((ops.layernorm_residual, P.layer_norm), (ops.rmsnorm_residual, lambda t, ww, e: P.unit_rms(t, e) * ww)):
        x = x0.clone()
        op(a, w, 1e-5, x, next_out=rounded)
        close(x, d64(x0) + plain(d64(a), d64(w), 1e-5), "float32", "stream after the norm")
        assert torch.equal(rounded, x.to(act(dtype)))
    # the mean of two normed sublayers, alone and into the norm
    mean = 0.5 * (P.unit_rms(d64(a), 1e-5) * d64(wa) + P.unit_rms(d64(b), 1e-5) * d64(wb))
    y = torch.zeros(rows, width, device=DEV)
    ops.pair_mean(a, wa, b, wb, 1e-5, y=y)
    close(y, mean, "float32", "mean of two")
    x = x0.clone()
    ops.pair_mean(a, wa, b, wb, 1e-5, norm_weight=w, norm_eps=1e-6, x=x, rounded=rounded)
    close(x, d64(x0) + P.layer_norm(mean, d64(w), 1e-6), "float32", "stream after the mean's norm")
    assert torch.equal(rounded, x.to(act(dtype)))
    x = x0.clone()
    ops.pair_mean(a, wa, b, wb, 1e-5, norm_weight=w, norm_eps=1e-6, x=x)
    close(x, d64(x0) + P.layer_norm(mean, d64(w), 1e-6), "float32", "without rounded rows")


@pytest.mark.parametrize("activation", ["relu2", "tanh"])
@pytest.mark.parametrize("m", [1, 8, 16, 40, 128, 300, 1100])
@pytest.mark.parametrize("width,cols", [(256, 320), (512, 1408), (64, 16), (1536, 512), (50, 36)])
def test_activation_of_a_products_outputs(m, width, cols, activation):
    """The serving precision applies it in the product's epilogue; the bits are those of the float32 product followed by the
    stand-alone kernel, for steps of few rows, of a tile's rows, of many tiles, and where rows do not start on 16 bytes."""
    g = torch.Generator().manual_seed(m + cols)
    x = torch.randn(m, width, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(cols, width, generator=g) * 1.5 / math.sqrt(width)).to(torch.bfloat16).to(DEV)
    ref = d64(x) @ d64(w).T
    ref = torch.relu(ref) ** 2 if activation == "relu2" else torch.tanh(ref)
    ops = ops_of("bfloat16")
    fused = torch.zeros(m, cols, dtype=torch.bfloat16, device=DEV)
    ops.linear(x, w, fused, activation=activation)
    y = torch.zeros(m, cols, device=DEV)
    ops.linear(x, w, y)
    apart = torch.zeros(m, cols, dtype=torch.bfloat16, device=DEV)
    ops.activate_rows(y, apart, activation)
    assert torch.equal(fused, apart)
    close(fused, ref, "bfloat16", activation)
    plain = torch.zeros(m, cols, dtype=torch.bfloat16, device=DEV)
    ops.linear(x, w, plain)                                        # and without one the product is still itself
    assert torch.equal(plain, y.to(torch.bfloat16))
    ops = ops_of("float32")
    out = torch.zeros(m, cols, device=DEV)
    ops.linear(x.float(), w.float(), out, activation=activation)
    close(out, ref, "float32", activation)
    ops_of("bfloat16").activate_rows(y[:, 3:9], apart[:, :6].contiguous())    # columns of wider rows, rounded only


# ---- attention inside chunks -----------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,dims", [(4, 2, 16, 16, 8), (3, 3, 10, 6, 4), (6, 1, 64, 32, 64), (2, 2, 200, 24, 130), (2, 1, 36, 12, 2)])
def test_biases_norms_and_the_half_layout_on_the_way_into_the_pages(dtype, heads, kv_heads, dim, vdim, dims):
    from bitwise_b200.parts.rope import HalfRotaryEncoding, LinearScaling
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(dim)
    seqs = [(0, 5), (37, 4), (250, 1), (15, 20)]
    b = Batch(seqs)
    page = 16
    table = scattered_table(seqs, page, g)
    cos, sin = HalfRotaryEncoding(dims, 300.0, LinearScaling(4.0), positions=300).rotary_tables(DEV)
    cols = heads * dim + kv_heads * (dim + vdim)
    wide = torch.randn(b.n, cols + 8, generator=g).to(DEV)
    u = wide[:, :cols]                                             # columns of a wider product
    bias = torch.randn(cols, generator=g).to(DEV)
    qn, kn = ((1.0 + 0.2 * torch.randn(dim, generator=g)).to(DEV) for _ in range(2))
    pages = int(table.max()) + 1
    kc = torch.zeros(pages, kv_heads, page, dim, dtype=act(dtype), device=DEV)
    vc = torch.zeros(pages, kv_heads, page, vdim, dtype=act(dtype), device=DEV)
    q = torch.zeros(b.n, heads * dim, dtype=act(dtype), device=DEV)
    ops.qkv_prepare(u, None, None, qn, kn, 1e-5, cos, sin, b, table, kc, vc, q, heads, kv_heads, dim, vdim, bias=bias, half_layout=True)
    y = d64(u) + d64(bias)
    rot = {"dims": dims, "base": 300.0, "scaling": {"factor": 4.0}}
    turned = lambda t, w: P.rotate_half(P.unit_rms(t.reshape(b.n, -1, dim), 1e-5) * d64(w), b.positions, rot)
    close(q, turned(y[:, :heads * dim], qn).reshape(b.n, -1), dtype, "queries")
    rows = lambda c: torch.stack([c[int(table[int(b.row_seq[r]), p // page]), :, p % page] for r, p in enumerate(b.positions)])
    close(rows(kc), turned(y[:, heads * dim:(heads + kv_heads) * dim], kn), dtype, "stored keys")
    close(rows(vc), y[:, (heads + kv_heads) * dim:].reshape(b.n, kv_heads, vdim), dtype, "stored values")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 32, 16), (3, 3, 10, 6), (8, 1, 64, 64)])
@pytest.mark.parametrize("chunk", [1, 7, 16, 40, 256, 300, 512, 2000])
def test_a_key_at_the_edges_of_a_chunk_and_far_inside_it(dtype, heads, kv_heads, dim, vdim, chunk):
    """Keys at the first position of every chunk, and just before it, point along the queries, so that they would carry the
    weight where they are seen: rows of prompts' portions and single rows, at chunk, page, key-tile and span edges.  Pages that
    only earlier chunks need hold rubbish."""
    ops = ops_of(dtype)
    g = torch.Generator().manual_seed(heads * dim + chunk)
    page, T = 16, 720
    table = scattered_table([(0, T), (0, T)], page, g)
    pages = int(table.max()) + 1
    kc = torch.zeros(pages, kv_heads, page, dim, dtype=act(dtype), device=DEV)
    vc = torch.zeros(pages, kv_heads, page, vdim, dtype=act(dtype), device=DEV)
    keys, vals = torch.randn(2, T, kv_heads, dim, generator=g) * 0.4, torch.randn(2, T, kv_heads, vdim, generator=g)
    direction = torch.randn(dim, generator=g)
    direction /= direction.norm()
    for start in range(0, T, chunk):
        keys[:, start] = direction * 6.0
        if chunk > 2 and start:
            keys[:, start - 1] = direction * 9.0
    idx = torch.arange(T)
    for s in range(2):
        kc[table[s].long()[idx // page], :, idx % page] = keys[s].to(act(dtype)).to(DEV)
        vc[table[s].long()[idx // page], :, idx % page] = vals[s].to(act(dtype)).to(DEV)
    k64 = [kc[table[s].long()[idx // page], :, idx % page].to(F64).cpu() for s in range(2)]
    v64 = [vc[table[s].long()[idx // page], :, idx % page].to(F64).cpu() for s in range(2)]
    scale = 0.5
    edge = chunk * max(1, min(700, 650) // chunk) if chunk < 700 else 700
    for seqs in ([(max(0, edge - 20), 40), (3, 5)], [(edge, 1), (max(0, edge - 1), 1)], [(min(edge + 1, T - 1), 1), (255, 1)], [(0, 90), (256, 3)],
                 [(500, 200), (31, 2)]):
        seqs = [(p0, min(c, T - p0)) for p0, c in seqs]
        b = Batch(seqs)
        q = torch.randn(b.n, heads, dim, generator=g) * 0.2 + direction * 3.0
        qd = q.reshape(b.n, -1).to(act(dtype)).to(DEV)
        # a page that no row of the step needs holds rubbish
        k2, v2 = kc.clone(), vc.clone()
        for s, (p0, c) in enumerate(seqs):
            for blk in range(p0 // chunk * chunk // page):
                k2[int(table[s, blk])], v2[int(table[s, blk])] = 1e4, 1e4
        out = torch.zeros(b.n, heads * vdim, dtype=act(dtype), device=DEV)
        ops.scored_attention(qd, k2, v2, table, out, heads, kv_heads, dim, vdim, scale, 0.0, False, None, 0, b, chunk=chunk)
        q64 = d64(qd).view(b.n, heads, dim)
        want = []
        for r, p in enumerate(b.positions):
            s, lo = int(b.row_seq[r]), p // chunk * chunk
            kk = k64[s][lo:p + 1].repeat_interleave(heads // kv_heads, 1)
            vv = v64[s][lo:p + 1].repeat_interleave(heads // kv_heads, 1)
            w = torch.softmax(torch.einsum("hd,khd->hk", q64[r], kk) * scale, -1)
            want.append(torch.einsum("hk,khd->hd", w, vv).reshape(-1))
        close(out, torch.stack(want), dtype, f"rows {seqs}, chunks of {chunk}", factor=2.0)


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


# lengths around the pages' (16), the key tiles' and spans' (32, 256) and the chunks' edges of each configuration
LENGTHS = {"a": [70, 41, 5, 300, 64, 17, 1, 131], "b": [100, 9, 290, 1, 65, 33], "c": [40, 270, 3, 17, 132], "d": [50, 33, 2, 100]}


def requests_of(name):
    return {f"{name}-{i}": tokens(CONFIGS[name], n, i) for i, n in enumerate(LENGTHS[name])}


def row_errors(got, want):
    """Per position: root mean square of the difference over that of the reference row."""
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean(-1))


def assess(errors, dtype, what, rounding_alone=None):
    """float32: every position within the tolerance.  bfloat16: against the errors that rounding alone causes in the
    plain implementation for the same weights and tokens (``rounding_alone``, per position)."""
    errors = np.concatenate([np.atleast_1d(e) for e in errors])
    if dtype == "float32":
        assert errors.max() <= 4 * TOL[dtype], f"{what}: worst relative error {errors.max():.3g}"
        return
    base = np.concatenate([np.atleast_1d(e) for e in rounding_alone])
    assert len(base) == len(errors)
    q = lambda e: float(np.quantile(e, 0.95))
    assert errors.mean() <= 2 * base.mean() + 0.01 and q(errors) <= 2 * q(base) + 0.02 and errors.max() <= 3 * base.max() + 0.05, \
        f"{what}: mean relative error {errors.mean():.3g} (rounding alone: {base.mean():.3g}), 95th percentile " \
        f"{q(errors):.3g} ({q(base):.3g}), worst {errors.max():.3g} ({base.max():.3g})"


def compare(name, dtype, got_by_request):
    errors, base = [], []
    for rid, toks in requests_of(name).items():
        want, rounded_ = plain_logits(name, toks, rounded_too=True)
        got = got_by_request[rid]
        assert got.shape == want.shape
        errors.append(row_errors(got, want))
        base.append(row_errors(rounded_, want))
    assess(errors, dtype, f"{name} {dtype} against the plain implementation", base)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
                b.forward = lambda ctx, x, cache, _o=orig: (_o(ctx, x, cache), caught.append(x.detach().clone()))
            make_replay_stepper(model, 384, use_graphs=False).run([StepEntry("r", toks, [])])
        finally:
            for b in model.decoder.blocks:
                del b.forward
        assert len(caught) == len(want)                      # a layer that runs another's block counts as well
        for i, (got, w) in enumerate(zip(caught, want)):
            close(got, w, "float32", f"stream after layer {i}", factor=4.0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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


def chunk_model(dtype, size):
    """One layer whose left attention alone is heard, with query and key projections that pass the first channels on: a
    token whose embedding is large along one channel is looked for by another such token."""
    from bitwise_b200 import Model
    cfg = ZuzupelConfig(vocab=40, width=32, eps=1e-5, layers=(
        L(pair(heads=2, kv_heads=1, dim=16, vdim=16, scale=1.5, dims=0, chunk=size, m_heads=1, m_dim=8, m_vdim=8, cap=4.0), 24),))
    W = random_weights(cfg, 5)
    p = "l0.mix.left."
    eye = torch.zeros(16, 32)
    eye[:, :16] = torch.eye(16)
    W[p + "q"], W[p + "k"] = torch.cat([eye, eye]).to(torch.bfloat16), eye.to(torch.bfloat16)
    for n in ("q.b", "k.b"):
        W[p + n] = torch.zeros_like(W[p + n])
    for n in ("q.norm", "k.norm"):
        W[p + n] = torch.ones_like(W[p + n])
    W["l0.mix.right.out"] = torch.zeros_like(W["l0.mix.right.out"])
    for t in (38, 39):
        W["embed"][t] = W["embed"][t] * 0.05
        W["embed"][t, 0] = 1.0
    return cfg, W, Model.from_tensors(cfg, W, dtype=dtype, device=DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("size", [24, 16, 33, 130])
def test_a_key_just_inside_and_just_outside_the_chunk(dtype, size):
    cfg, W, model = chunk_model(dtype, size)
    total = 200
    start = (total - 1) // size * size                        # the last position's chunk begins here
    base = [t % 38 for t in tokens(cfg, total, 1)]
    plain = list(base)
    plain[-1] = 39
    unmarked = P.forward(cfg.to_json(), W, plain)[-1].numpy()
    for tail in (0, total - start + 3):                       # the last position in a prompt's portion, and decoded alone
        outs = {}
        for at in (start, start - 1):
            toks = list(plain)
            toks[at] = 38
            want, rounded_ = plain_pair(cfg, W, toks)
            steps = R.tail_one_by_one({"r": toks}, tail=tail) if tail else R.portions({"r": toks}, sizes=(61, 2, 90, 47))
            got = R.collect(steps, R.run_in_process(model, steps, 256), cfg.vocab)["r"]
            assess([row_errors(got, want)], dtype, f"marked key at {at}", [row_errors(rounded_, want)])
            outs[at] = (want[-1], got[-1])
        (want_in, got_in), (want_out, got_out) = outs[start], outs[start - 1]
        assert np.abs(want_out - unmarked).max() < 1e-9 * np.abs(unmarked).max() + 1e-9, "a key outside the chunk changed the logits"
        assert np.abs(want_in - unmarked).max() > 0.04 * np.abs(unmarked).max(), "the key inside the chunk did not decide"
        gap = np.abs(want_in - want_out).max()
        assert np.abs(got_in - want_in).max() < 0.25 * gap and np.abs(got_out - want_out).max() < 0.25 * gap


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_over_reused_pages(dtype):
    # one request decoded token by token from position 3 to past 500 (pages, key tiles, spans and chunks are crossed one
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_simulated_traces_reproduce_requests_run_alone(dtype):
    # the engine's simulator: random requests, budgets and pools, preemption with recomputation; a request's tokens
    # and the fingerprint of its logits must be those it yields alone on an idle engine
    from bitwise_b200.engine.simulate import run_traces
    out = run_traces(model_of("a", dtype), traces=8, seed=5)
    assert out.traces == 8 and out.requests_checked > 10
    assert out.violations == 0, (out.token_mismatch, out.fingerprint_mismatch, out.hangs, out.leaks)


def test_command_line_random_folder_replay_and_generation(tmp_path):
    """``bitwise_b200 random`` writes a Zuzupel folder from a config.json; ``bin/trace_run`` replays a mixed schedule
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
