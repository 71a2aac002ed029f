"""Small Sazisun configurations for the tests, and weights for them.

The configurations differ from one another in every size and in the order of their layers: widths that are no multiple
of 8, one head and many, maps that share a key head, value sizes below and above a warp's lanes, partly turned maps with and
without a rescaling, scores with and without a cap, layers that read another's keys (two of one layer, with other constants),
convolutions of one to six taps, states below and above a warp's lanes, every kind of feed-forward and none.

Weights are drawn so that scores, gates, decays and activations are of order one.  The experts' choice must not hang on
rounding: the first channels of the embedding hold well separated levels, one channel per expert, that no layer adds to, and
the router of a layer reads its experts' channels (in an order of its own).
"""
import numpy as np
import torch

from bitwise_b200.config.sazisun import (ExpertsConfig, FeedForwardConfig, SazisunConfig, SazisunLayerConfig, StateSpaceConfig,
                                         TwoMapAttentionConfig, WavelengthScalingConfig)

L = SazisunLayerConfig
SCALING = WavelengthScalingConfig(factor=3.0, low=1.5, high=6.0, original=90.0)


def attention(heads=4, kv_heads=2, dim=16, vdim=32, scale=0.3, diff=0.35, softcap=6.0, base=3000.0, dims=8, scaling=SCALING, kv_from=None):
    return TwoMapAttentionConfig(heads, kv_heads, dim, vdim, scale, diff, softcap, base if dims else None, dims or None,
                                 scaling if dims else None, kv_from)


def space(heads=6, vdim=16, state=24, groups=3, conv=4, norm_groups=2):
    return StateSpaceConfig(heads, vdim, state, groups, conv, norm_groups)


def experts(ff=24, experts=6, top=2, scale=1.7, groups=3, keep_groups=2, shared_ff=40):
    return ExpertsConfig(ff, experts, top, scale, groups, keep_groups, shared_ff)


D = FeedForwardConfig
CONFIGS = {
    # every branch; the tensor-core kernels take these shapes on the serving precision
    "a": SazisunConfig(vocab=149, width=80, eps=1e-5, layers=(
        L(attention(), D(112)),
        L(space(), experts()),
        L(attention(scale=0.5, diff=0.7, softcap=None, kv_from=0), None),
        L(attention(heads=6, kv_heads=3, dim=32, vdim=48, dims=32, base=500.0, scaling=None), experts(ff=32, experts=8, top=3, groups=4, keep_groups=2,
                                                                                                      shared_ff=None, scale=0.8)),
        L(space(heads=2, vdim=32, state=16, groups=1, conv=3, norm_groups=1), experts(ff=16, groups=1, keep_groups=1, top=1, shared_ff=16)))),
    # odd sizes everywhere, one key head, one tap (no convolution state), no cap
    "b": SazisunConfig(vocab=97, width=50, eps=1e-6, layers=(
        L(space(heads=5, vdim=9, state=7, groups=1, conv=1, norm_groups=3), D(36)),
        L(attention(heads=3, kv_heads=1, dim=10, vdim=7, scale=0.8, diff=0.2, softcap=None, base=50.0, dims=6, scaling=None),
          experts(ff=9, experts=5, top=5, groups=1, keep_groups=1, scale=1.0, shared_ff=13)),
        L(attention(heads=3, kv_heads=1, dim=10, vdim=7, scale=0.4, diff=0.9, softcap=3.0, base=50.0, dims=6, scaling=None, kv_from=1),
          experts(ff=20, experts=7, top=2, groups=7, keep_groups=3, shared_ff=5)),
        L(space(heads=3, vdim=5, state=11, groups=3, conv=2, norm_groups=5), None))),
    # heads beyond the tensor-core kernel, a state beyond 128, long taps, two layers on one layer's keys, no rotation
    "c": SazisunConfig(vocab=64, width=48, eps=1e-5, layers=(
        L(space(heads=2, vdim=20, state=140, groups=2, conv=6, norm_groups=1), D(40)),
        L(attention(heads=2, kv_heads=2, dim=72, vdim=144, scale=0.12, diff=0.5, softcap=30.0, dims=0), None),
        L(attention(heads=2, kv_heads=2, dim=72, vdim=144, scale=0.2, diff=0.1, softcap=9.0, dims=0, kv_from=1), D(24)),
        L(attention(heads=2, kv_heads=2, dim=72, vdim=144, scale=0.1, diff=0.3, softcap=None, dims=0, kv_from=1), experts(experts=4, groups=2, keep_groups=1)),
        L(space(heads=4, vdim=64, state=36, groups=2, conv=5, norm_groups=8), None))),
    # no pages at all
    "d": SazisunConfig(vocab=40, width=32, eps=1e-5, layers=(
        L(space(heads=2, vdim=16, state=16, groups=2, conv=3, norm_groups=2), D(24)),
        L(space(heads=4, vdim=8, state=12, groups=1, conv=4, norm_groups=4), experts(experts=4, groups=2, keep_groups=1, top=2)))),
}


def random_weights(config, seed, std=None):
    """name -> bfloat16 CPU tensor."""
    from bitwise_b200.config.registry import lookup_architecture
    g = torch.Generator().manual_seed(seed)
    specs = lookup_architecture("Sazisun").build(config).param_specs()
    routed = {f"l{i}": l.mlp for i, l in enumerate(config.layers) if l.mlp is not None and l.mlp.kind == "moe"}
    marks = max([m.experts for m in routed.values()], default=0)   # the channels that the routers read
    r = lambda *s: torch.randn(*s, generator=g)
    out = {}
    for s in specs:
        n = s.name
        if n.endswith(".A_log"):
            t = r(*s.shape) * 0.7 - 0.5
        elif n.endswith(".dt_bias"):
            t = r(*s.shape) - 1.5
        elif n.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = r(*s.shape) * 0.8 / s.shape[0] ** 0.25
        elif n.endswith(".alpha"):
            t = 0.4 + 0.3 * torch.rand((), generator=g)
        elif n.endswith((".norm1", ".norm2", "final.norm")):
            t = 1.0 + 0.2 * r(*s.shape)
            t[:marks] = 1.0
        elif n.endswith((".norm1.b", ".norm2.b", "final.norm.b")):
            t = 0.2 * r(*s.shape)
            t[:marks] = 0.0
        elif n.endswith(".conv"):
            t = r(*s.shape) * 0.6
        elif n.endswith(".conv.b"):
            t = r(*s.shape) * 0.3
        elif n.endswith(".D") or n.endswith(".mix.norm"):
            t = 1.0 + 0.3 * r(*s.shape)
        elif n == "embed":
            t = r(*s.shape)
            if marks:
                levels = torch.linspace(-1.6, 1.6, marks)
                t[:, :marks] = levels[torch.argsort(torch.rand(s.shape[0], marks, generator=g), 1)]
        elif n.endswith(".router"):
            m = routed[n.split(".")[0]]
            t = 0.01 * r(*s.shape)
            t[torch.arange(m.experts), torch.randperm(marks, generator=g)[:m.experts]] += 4.0
        else:
            t = r(*s.shape) * (std or 0.8 / np.sqrt(s.shape[1]))
            if n.endswith((".mix.o", ".down")):
                t[:marks] = 0.0
        out[n] = t.to(torch.bfloat16)
    return out


def tokens(config, n, seed):
    return np.random.default_rng(seed).integers(0, config.vocab, n).tolist()
