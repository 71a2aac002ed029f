"""The Sazisun design stated plainly: whole sequences, no cache, no batching, float64 on the CPU.

One function per mechanism, written from the design's equations and sharing nothing with the
package: the tests compare the package's kernels, cache, state and scheduler with these.

Notation: x is [tokens, width]; a weight W is stored [out, in] and applied as ``x @ W.T``; ``w``
is a dict name -> tensor; ``cfg`` is the model's config.json as a dict; S is a head's matrix of
state, [state, vdim].

* a layer is ``x += mixer(norm1(x))``, ``x += ff(norm2(x))`` with ``norm(x) = tanh(alpha x) w + b``
* two-map attention: two softmaxes per head over the same values, ``a1 - lambda a2``, a norm over the head, a gate
* state space: ``S <- e^(-rate dt) S + dt B x^T``, ``y = S^T C + D x``, a gate, a norm over groups of entries
* the feed-forward is gated (SiLU), or routed over experts ``W_down relu(W_up h)^2`` with a gated shared one
"""
import contextlib
import math

import torch

F64 = torch.float64

_ROUND = None


@contextlib.contextmanager
def rounding(fn):
    """Inside the block, what the serving precision stores in 16 bits between its kernels (the products' inputs, cached
    keys and values) is passed through ``fn``: the plain result then shows how large an error rounding alone causes."""
    global _ROUND
    _ROUND, old = fn, _ROUND
    try:
        yield
    finally:
        _ROUND = old


def stored(x):
    return _ROUND(x) if _ROUND is not None else x


def tanh_norm(x, alpha, g, b):
    return torch.tanh(alpha * x) * g + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


# ---- the state-space mixer -------------------------------------------------------------------------------
def causal_conv(u, taps_w, bias):
    """u: [tokens, channels]; taps_w: [channels, taps]; y_t = bias + sum_j w[:, j] u_(t - taps + 1 + j)."""
    n, taps = u.shape[0], taps_w.shape[1]
    y = torch.zeros_like(u) + bias
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] += taps_w[:, j] * u[:n - back]
    return y


def step_sizes(z, bias):
    return softplus(z + bias)


def space_scan(x, B, C, dt, rate, D, S=None):
    """x: [tokens, heads, vdim]; B, C: [tokens, heads, state]; dt: [tokens, heads]; rate, D: [heads].  Returns the outputs
    and the last state, one token after the other."""
    n, H, vd = x.shape
    S = torch.zeros(H, B.shape[2], vd, dtype=F64) if S is None else S.clone()
    out = []
    for t in range(n):
        S = torch.exp(-rate * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t])
    return torch.stack(out), S


def gated_group_norm(y, z, g, groups, eps):
    """The gate first, then a norm of every one of ``groups`` equal parts of the row by itself."""
    y = y * silu(z)
    parts = y.reshape(y.shape[0], groups, -1)
    return unit_rms(parts, eps).reshape(y.shape) * g


def space_mixer(h, w, pre, c, eps):
    n = h.shape[0]
    H, vd, N, G = c["heads"], c["vdim"], c["state"], c["groups"]
    inner = H * vd
    u = h @ w[pre + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x = xbc[:, :inner].reshape(n, H, vd)
    B = xbc[:, inner:inner + G * N].reshape(n, G, N).repeat_interleave(H // G, 1)
    C = xbc[:, inner + G * N:].reshape(n, G, N).repeat_interleave(H // G, 1)
    y, _ = space_scan(x, B, C, step_sizes(dt, w[pre + "dt_bias"]), torch.exp(w[pre + "A_log"]), w[pre + "D"])
    y = gated_group_norm(y.reshape(n, inner), z, w[pre + "norm"], c["norm_groups"], eps)
    return stored(y) @ w[pre + "o"].T


# ---- two-map attention -----------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """base^(-2i/dims), rescaled by wavelength: short ones stay, long ones are divided by the factor, between a blend."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(v, positions, rot):
    """v: [tokens, ..., n]; of the first ``dims`` entries, 2i and 2i + 1 turn together; the rest pass."""
    out = v.clone()
    p = torch.as_tensor(positions, dtype=F64).reshape((-1,) + (1,) * (v.dim() - 2))
    for i, f in enumerate(rotary_frequencies(rot)):
        c, s = torch.cos(p * f), torch.sin(p * f)
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = a * c - b * s
        out[..., 2 * i + 1] = b * c + a * s
    return out


def capped_attention(q, k, v, scale, cap):
    """q, k: [tokens, heads, dim]; v: [tokens, heads, vdim]; every position sees itself and what came before."""
    n = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    s = s.masked_fill(torch.ones(n, n).triu(1).bool()[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def subtraction_weight(w, pre, diff):
    return torch.exp((w[pre + "lq1"] * w[pre + "lk1"]).sum()) - torch.exp((w[pre + "lq2"] * w[pre + "lk2"]).sum()) + diff


def subtract_and_norm(a1, a2, lam, diff, eps):
    """[tokens, heads, vdim] each."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def two_map_attention(h, w, pre, c, eps, positions, kept=None):
    """Returns the mixer's output and the keys and values as a later layer may use them (``kept``: such a pair)."""
    n = h.shape[0]
    H, G, dim, vd = c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def turned(t):
        return stored(rotate_pairs(t, positions, c["rot"]) if c.get("rot") else t)

    q = turned((h @ w[pre + "q"].T).reshape(n, H, 2, dim))
    if kept is None:
        kept = (turned((h @ w[pre + "k"].T).reshape(n, G, 2, dim)), stored((h @ w[pre + "v"].T).reshape(n, G, vd)))
    k, v = (t.repeat_interleave(H // G, 1) for t in kept)
    a1, a2 = (capped_attention(q[:, :, m], k[:, :, m], v, c["scale"], c.get("softcap")) for m in range(2))
    o = subtract_and_norm(a1, a2, subtraction_weight(w, pre, c["diff"]), c["diff"], eps).reshape(n, H * vd)
    return stored(o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T, kept


# ---- feed-forward ----------------------------------------------------------------------------------------
def gated_ff(h, w, pre):
    return stored(silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def expert(h, w, pre):
    a = torch.relu(h @ w[pre + "up"].T)
    return stored(a * a) @ w[pre + "down"].T


def choose(z, r):
    """Router logits of one token -> (experts in the order of choice, weights)."""
    E, top = r["experts"], r["top"]
    s = torch.softmax(z, -1)
    groups = r.get("groups") or {"count": 1, "keep": 1}
    per = E // groups["count"]
    best = sorted(range(groups["count"]), key=lambda j: (-float(s[j * per:(j + 1) * per].max()), j))[:groups["keep"]]
    allowed = [e for e in range(E) if e // per in best]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    ws = s[chosen] / (s[chosen].sum() + 1e-20) * r.get("scale", 1.0)
    return chosen, ws


def routed_ff(h, w, pre, c):
    out = torch.zeros_like(h)
    z = h @ w[pre + "router"].T
    for t in range(h.shape[0]):
        for e, wt in zip(*choose(z[t], c["router"])):
            out[t] += wt * expert(h[t], w, f"{pre}e{e}.")
    if c.get("shared"):
        out = out + torch.sigmoid(h @ w[pre + "shared.sg"].T) * expert(h, w, pre + "shared.")
    return out


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] of one whole sequence; ``layers_out``: a list that receives the stream after
    every layer."""
    w = {k: v.to(F64) for k, v in weights.items() if v.dtype != torch.int32}
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))

    def norm(x, name):
        return stored(tanh_norm(x, w[name + ".alpha"], w[name], w[name + ".b"]))

    x = w["embed"][torch.as_tensor(tokens)]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "mamba2":
            y = space_mixer(h, w, p + "mix.", c, eps)
        else:
            y, kept[i] = two_map_attention(h, w, p + "mix.", c, eps, positions, kept.get(c.get("kv_from")))
        x = x + y
        f = layer.get("mlp")
        if f:
            h = norm(x, p + "norm2")
            x = x + (routed_ff(h, w, p + "mlp.", f) if f["kind"] == "moe" else gated_ff(h, w, p + "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ w["embed"].T
