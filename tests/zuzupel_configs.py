"""Small Zuzupel configurations for the tests, and weights for them.

The configurations differ from one another in every size and in the order of their layers: widths that are no multiple
of 8, one head and many, key sizes below and above a warp's lanes, value sizes unlike the key sizes, query heads that share a
key head, convolutions of one to five taps, chunks shorter and longer than a page and than the prompts, partly turned
heads, layers that run another layer's weights, layers without feed-forward.  Weights are drawn so that scores, gates,
decays and activations are of order one.
"""
import numpy as np
import torch

from bitwise_b200.config.zuzupel import (ChannelDeltaConfig, ChunkAttentionConfig, MatrixMemoryConfig, ParallelConfig, WkvConfig,
                                         ZuzupelConfig, ZuzupelLayerConfig)

L = ZuzupelLayerConfig


def wkv(heads=3, dim=16, rank=8):
    return WkvConfig(heads, dim, decay_rank=rank)


def delta(heads=4, kv_heads=2, dim=16, vdim=16, conv=4, rank=8, gate_rank=12):
    return ChannelDeltaConfig(heads, kv_heads, dim, vdim, conv, decay_rank=rank, gate_rank=gate_rank)


def pair(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, base=10000.0, dims=8, factor=4.0, chunk=24, m_heads=3, m_dim=16,
         m_vdim=24, cap=8.0):
    return ParallelConfig(ChunkAttentionConfig(heads, kv_heads, dim, vdim, scale, base if dims else None, dims or None, factor if dims else None, chunk),
                          MatrixMemoryConfig(m_heads, m_dim, m_vdim, cap))


CONFIGS = {
    # every mixer; the tensor-core kernels take these shapes on the serving precision
    "a": ZuzupelConfig(vocab=149, width=64, eps=1e-5, layers=(
        L(pair(heads=4, kv_heads=2, dim=32, vdim=16, scale=0.3, base=5000.0, dims=32, factor=2.0, chunk=40, m_heads=2, m_dim=24,
               m_vdim=40, cap=5.0), 112),
        L(wkv(heads=3, dim=24, rank=10), 80),
        L(delta(heads=6, kv_heads=2, dim=16, vdim=32, conv=3, rank=9, gate_rank=20), None),
        L(pair(heads=2, kv_heads=1, dim=16, vdim=48, scale=0.5, base=300.0, dims=8, factor=8.0, chunk=16, m_heads=1, m_dim=40,
               m_vdim=16, cap=20.0), 48),
        L(delta(heads=6, kv_heads=2, dim=16, vdim=32, conv=3, rank=9, gate_rank=20), None, weights_of=2))),
    # odd sizes everywhere, one head, one tap (no convolution state), no rotation, no rescaling, no chunk; a wkv layer and a
    # parallel layer run a second time with a state of their own
    "b": ZuzupelConfig(vocab=97, width=50, eps=1e-6, layers=(
        L(delta(heads=1, kv_heads=1, dim=7, vdim=5, conv=1, rank=3, gate_rank=1), 36),
        L(wkv(heads=5, dim=9, rank=1), 28),
        L(pair(heads=3, kv_heads=3, dim=10, vdim=6, scale=1.1, dims=4, base=50.0, factor=None, chunk=None, m_heads=5, m_dim=6, m_vdim=3,
               cap=2.5), 20),
        L(wkv(heads=5, dim=9, rank=1), 28, weights_of=1),
        L(pair(heads=3, kv_heads=3, dim=10, vdim=6, scale=1.1, dims=4, base=50.0, factor=None, chunk=None, m_heads=5, m_dim=6, m_vdim=3,
               cap=2.5), 20, weights_of=2))),
    # large heads (every lane layout of the recurrences), a chunk of one page and of 7, value heads smaller than a block's
    # columns, long taps; the second layer's weights belong to a later one
    "c": ZuzupelConfig(vocab=64, width=48, eps=1e-5, layers=(
        L(delta(heads=2, kv_heads=1, dim=72, vdim=20, conv=5, rank=16, gate_rank=8), 40),
        L(wkv(heads=1, dim=40, rank=33), 24, weights_of=3),
        L(pair(heads=8, kv_heads=1, dim=8, vdim=8, scale=0.9, dims=0, chunk=7, m_heads=2, m_dim=140, m_vdim=4, cap=15.0), None),
        L(wkv(heads=1, dim=40, rank=33), 24),
        L(delta(heads=3, kv_heads=3, dim=36, vdim=64, conv=2, rank=4, gate_rank=40), None))),
    # no pages at all
    "d": ZuzupelConfig(vocab=40, width=32, eps=1e-5, layers=(
        L(wkv(heads=2, dim=16, rank=4), 24), L(delta(heads=2, kv_heads=2, dim=8, vdim=12, conv=4, rank=4, gate_rank=4), 24))),
}


def random_weights(config, seed, std=None):
    """name -> bfloat16 CPU tensor."""
    from bitwise_b200.config.registry import lookup_architecture
    g = torch.Generator().manual_seed(seed)
    specs = lookup_architecture("Zuzupel").build(config).param_specs()
    out = {}
    for s in specs:
        n = s.name
        if n.endswith(".A_log"):
            t = torch.randn(s.shape, generator=g) * 0.5 - 1.5
        elif n.endswith(".w0"):
            t = torch.randn(s.shape, generator=g) * 0.8 - 2.5       # decays from a half to nearly one
        elif n.endswith(".f.b"):
            t = torch.randn(s.shape, generator=g) + 2.0              # forget gates mostly open
        elif ".mu." in n:
            t = torch.rand(s.shape, generator=g)
        elif n.endswith((".u", ".b", ".dt_bias")) and len(s.shape) < 2 or n.endswith(".mix.u"):
            t = torch.randn(s.shape, generator=g) * 0.5
        elif n.endswith(".conv"):
            t = torch.randn(s.shape, generator=g) * 0.6
        elif len(s.shape) == 1:
            t = 1.0 + 0.2 * torch.randn(s.shape, generator=g)
        elif n == "embed":
            t = torch.randn(s.shape, generator=g)
        else:
            t = torch.randn(s.shape, generator=g) * (std or 0.8 / np.sqrt(s.shape[1]))
        out[n] = t.to(torch.bfloat16)
    return out


def tokens(config, n, seed):
    return np.random.default_rng(seed).integers(0, config.vocab, n).tolist()
