"""The Zuzupel design stated plainly: whole sequences, no cache, no batching, float64 on the CPU.

One function per mechanism, written from the design's equations and sharing nothing with the
package: the tests compare the package's kernels, cache, state and scheduler with these.

Notation: x is [tokens, width]; a weight W is stored [out, in] and applied as ``x @ W.T``; ``w``
is a dict name -> tensor; ``cfg`` is the model's config.json as a dict; S is a head's matrix of
state, [dim, vdim].

* a layer is ``x += norm1(mixer(x))``, ``x += norm2(ff(x))``, the norms layer norms without bias
* delta rule with a decay per key channel: ``S <- g S``, ``S <- S + k (beta (v - S^T k))^T``, ``o = S^T q``
* time mixing with a bonus for the current token: ``o = (S + diag(u) k v^T)^T r``, then ``S <- diag(w) S + k v^T``
* matrix memory with a running maximum: ``S <- e^(f + m' - m) S + e^(i - m) k v^T``, a normaliser beside it
* attention inside chunks, biased projections, a weighted norm per head, a half-layout rotation
* two mixers side by side, half the sum of their normed outputs
* the feed-forward is ``W_down relu(W_up h)^2``
"""
import contextlib
import math

import torch

F64 = torch.float64

_ROUND = None


@contextlib.contextmanager
def rounding(fn):
    """Inside the block, what the serving precision stores in 16 bits between its kernels (the products' inputs, cached
    keys and values, the heads' outputs) is passed through ``fn``: the plain result then shows how large an error
    rounding alone causes."""
    global _ROUND
    _ROUND, old = fn, _ROUND
    try:
        yield
    finally:
        _ROUND = old


def stored(x):
    return _ROUND(x) if _ROUND is not None else x


def layer_norm(x, g, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * g


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x, eps=1e-6):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def log_sigmoid(z):
    return -softplus(-z)


def causal_conv(u, taps_w):
    """u: [tokens, channels]; taps_w: [channels, taps]; y_t = sum_j w[:, j] u_(t - taps + 1 + j)."""
    n, taps = u.shape[0], taps_w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] += taps_w[:, j] * u[:n - back]
    return y


def previous_rows(h):
    """Row t holds row t - 1 of h; zeros before the start."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]], 0)


# ---- the three recurrences, one token after the other; every input [tokens, heads, size] -----------------
def delta_scan(q, k, v, g, beta, S=None):
    """g: decay per head and key channel; beta: [tokens, heads].  Returns the outputs and the last state."""
    n, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=F64) if S is None else S.clone()
    out = []
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def bonus_scan(r, k, v, w, u, S=None):
    """w: decay per head and key channel; u: [heads, dim], the current token's bonus."""
    n, H, dim = r.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=F64) if S is None else S.clone()
    out = []
    for t in range(n):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t]))
        S = w[t][:, :, None] * S + kv
    return torch.stack(out), S


def matrix_memory_scan(q, k, v, i, f, S=None, nrm=None, m=None):
    """i, f: [tokens, heads], the logarithms of the input and the forget gate.  q arrives scaled."""
    n, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=F64) if S is None else S.clone()
    nrm = torch.zeros(H, dim, dtype=F64) if nrm is None else nrm.clone()
    m = torch.zeros(H, dtype=F64) if m is None else m.clone()
    out = []
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * (k[t][:, :, None] * v[t][:, None, :])
        nrm = keep[:, None] * nrm + add[:, None] * k[t]
        m = new
        den = torch.maximum((nrm * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None])
    return torch.stack(out), (S, nrm, m)


# ---- the mixers ------------------------------------------------------------------------------------------
def delta_mixer(h, w, pre, c, eps):
    n = h.shape[0]
    H, G, dim, vd = c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def project(name):
        return silu(causal_conv(h @ w[pre + name].T, w[pre + name + ".conv"]))

    q = unit_length(project("q").reshape(n, G, dim)) * dim ** -0.5
    k = unit_length(project("k").reshape(n, G, dim))
    v = project("v").reshape(n, H, vd)
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    z = stored(h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]
    g = torch.exp(-torch.exp(w[pre + "A_log"])[None, :, None] * softplus(z).reshape(n, H, dim))
    o, _ = delta_scan(q, k, v, g, beta)
    gate = torch.sigmoid(stored(h @ w[pre + "g1"].T) @ w[pre + "g2"].T).reshape(n, H, vd)
    o = unit_rms(o, eps) * w[pre + "norm"] * gate
    return stored(o.reshape(n, H * vd)) @ w[pre + "o"].T


def wkv_mixer(x, w, pre, c, eps):
    """x: the stream itself, before rounding (the mixes are formed in full precision)."""
    n = x.shape[0]
    H, dim = c["heads"], c["dim"]
    shift = previous_rows(x) - x
    mix = {s: stored(x + shift * w[pre + "mu." + s]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[pre + s].T).reshape(n, H, dim) for s in "rkv")
    gate = silu(mix["g"] @ w[pre + "g"].T)
    z = stored(torch.tanh(mix["w"] @ w[pre + "w1"].T)) @ w[pre + "w2"].T + w[pre + "w0"]
    decay = torch.exp(-torch.exp(z)).reshape(n, H, dim)
    o, _ = bonus_scan(r, k, v, decay, w[pre + "u"])
    o = unit_rms(o, eps).reshape(n, H * dim) * w[pre + "norm"] * gate
    return stored(o) @ w[pre + "o"].T


def memory_mixer(h, w, pre, c, eps):
    n = h.shape[0]
    H, dim, vd, cap = c["heads"], c["dim"], c["vdim"], c["gate_cap"]
    q = (h @ w[pre + "q"].T).reshape(n, H, dim) * dim ** -0.5
    k = (h @ w[pre + "k"].T).reshape(n, H, dim)
    v = (h @ w[pre + "v"].T).reshape(n, H, vd)
    i = cap * torch.tanh((h @ w[pre + "i"].T + w[pre + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ w[pre + "f"].T + w[pre + "f.b"]) / cap))
    o, _ = matrix_memory_scan(q, k, v, i, f)
    o = unit_rms(o, eps).reshape(n, H * vd) * w[pre + "norm"] * torch.sigmoid(h @ w[pre + "g"].T)
    return stored(o) @ w[pre + "o"].T


def rotary_frequencies(rot):
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate_half(v, positions, rot):
    """v: [tokens, ..., n]; of the first ``dims`` entries, i and i + dims / 2 turn together; the rest pass."""
    half = int(rot["dims"]) // 2
    out = v.clone()
    p = torch.as_tensor(positions, dtype=F64).reshape((-1,) + (1,) * (v.dim() - 2))
    for i, f in enumerate(rotary_frequencies(rot)):
        c, s = torch.cos(p * f), torch.sin(p * f)
        a, b = v[..., i], v[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


def chunk_visible(positions, size):
    """[i, j]: whether position i sees position j (every earlier one where there are no chunks)."""
    p = torch.as_tensor(positions)
    seen = p[None, :] <= p[:, None]
    if size:
        seen = seen & (p[None, :] // size == p[:, None] // size)
    return seen


def chunk_attention(h, w, pre, c, eps, positions):
    n = h.shape[0]
    H, G, dim, vd = c["heads"], c["kv_heads"], c["dim"], c["vdim"]

    def project(name, heads, size):
        return (h @ w[pre + name].T + w[pre + name + ".b"]).reshape(n, heads, size)

    q = unit_rms(project("q", H, dim), eps) * w[pre + "q.norm"]
    k = unit_rms(project("k", G, dim), eps) * w[pre + "k.norm"]
    v = stored(project("v", G, vd))
    if c.get("rot"):
        q, k = rotate_half(q, positions, c["rot"]), rotate_half(k, positions, c["rot"])
    q, k = stored(q), stored(k)
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * c["scale"]
    s = s.masked_fill(~chunk_visible(positions, (c.get("mask") or {}).get("size"))[None], -math.inf)
    o = torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)
    return stored(o.reshape(n, H * vd)) @ w[pre + "o"].T


def parallel_mixer(h, w, pre, c, eps, positions):
    left = chunk_attention(h, w, pre + "left.", c["left"], eps, positions)
    right = memory_mixer(h, w, pre + "right.", c["right"], eps)
    return 0.5 * (unit_rms(left, eps) * w[pre + "left.out"] + unit_rms(right, eps) * w[pre + "right.out"])


def dense_ff(h, w, pre):
    a = torch.relu(h @ w[pre + "up"].T)
    return stored(a * a) @ w[pre + "down"].T


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [tokens, vocab] of one whole sequence; ``layers_out``: a list that receives the stream after
    every layer."""
    w = {k: v.to(F64) for k, v in weights.items() if v.dtype != torch.int32}
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens)))
    x = w["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i if layer.get('weights_of') is None else layer['weights_of']}."
        c = layer["mixer"]
        if layer["type"] == "wkv":
            y = wkv_mixer(x, w, p + "mix.", c, eps)
        elif layer["type"] == "channel_delta":
            y = delta_mixer(stored(x), w, p + "mix.", c, eps)
        else:
            y = parallel_mixer(stored(x), w, p + "mix.", c, eps, positions)
        x = x + layer_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(dense_ff(stored(x), w, p + "mlp."), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return stored(layer_norm(x, w["final.norm"], eps)) @ w["head"].T
