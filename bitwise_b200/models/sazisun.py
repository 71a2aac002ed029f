"""Sazisun assembled from parts, and its entry in the architecture registry.

A decoder of pre-norm blocks, ``x += mixer(norm1(x))``, ``x += ff(norm2(x))``, whose norms compute no statistics (``TanhNorm``).
Two kinds of mixer, in any order:

* ``attention``: two maps per head over the same values whose outputs are subtracted, capped scores, a rotation of the leading
  entries of every map with frequencies rescaled by wavelength, a norm per head and an output gate
  (``ScoredAttention(difference=)``); a layer may read the keys and values of an earlier one;
* ``mamba2``: a state-space recurrence behind a short convolution, its output gated and normed in groups (``StateSpace``).

The feed-forward is the dense gated one (SiLU), or routed: softmax scores over all experts, groups of experts of which the best
stay eligible by their largest score, weights divided by their sum, experts with the square of relu, and a shared expert behind
a sigmoid gate; or absent.  The head is the embedding table behind a last norm.

Tensor names: ``embed``, ``final.norm``, and per layer ``l<i>.norm1``, ``l<i>.norm2`` (each with ``.b`` and ``.alpha``), ``l<i>.mix.*``
(see the mixers), ``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.e<k>.{up, down}``, ``l<i>.mlp.router``, ``l<i>.mlp.shared.{up, down, sg}``.
Matrices are stored [out, in].
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sazisun import SazisunConfig
from ..parts.block import PreNormBlock, chain_norms
from ..parts.embedding import OutputHead, TokenEmbedding
from ..parts.mlp import DenseFFN, SwiGLU
from ..parts.norm import TanhNorm
from ..parts.rope import PairRotaryEncoding, WavelengthScaling
from ..parts.routed_ffn import RoutedFFN
from ..parts.scored_attention import ScoredAttention
from ..parts.state_recurrence import StateSpace
from .decoder import DecoderModel, LayerRun

BLOCK_NAMES = {"mixer_norm": "norm1", "mixer": "mix", "ffn_norm": "norm2", "feed_forward": "mlp"}
WEIGHT_SUM_EPS = 1e-20  # joins the sum that the chosen experts' scores are divided by


def build_sazisun(config: SazisunConfig) -> DecoderModel:
    c = config
    rotaries = {}   # one table per (turned entries, base, rescaling)

    def mixer_of(m):
        if m.kind == "mamba2":
            return StateSpace(c.width, m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups, c.eps)
        rotary = None
        if m.rot_dims:
            key = (m.rot_dims, m.rot_base, m.rot_scaling)
            if key not in rotaries:
                s = m.rot_scaling
                rotaries[key] = PairRotaryEncoding(m.rot_dims, m.rot_base,
                                                   WavelengthScaling(s.factor, s.low, s.high, s.original) if s else None)
            rotary = rotaries[key]
        return ScoredAttention(c.width, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, c.eps, position=rotary, rot_dims=m.rot_dims or 0,
                               softcap=m.softcap, shares_cache=m.kv_from is not None, gate="entry", difference=m.diff)

    def feed_forward_of(f):
        if f is None:
            return None
        if f.kind == "dense":
            return SwiGLU(c.width, f.ff, names=("gate", "up", "down"), suffix="")
        shared = DenseFFN(c.width, f.shared_ff) if f.shared_ff else None
        return RoutedFFN(c.width, f.experts, f.top, f.ff, 0.0, 0.0, f.scale, f.groups, f.keep_groups, correction=False, shared=shared,
                         scoring="softmax", activation="relu2", group_score="max", sum_eps=WEIGHT_SUM_EPS,
                         shared_gate="shared.sg" if shared else None)

    blocks, schedule, entry_of = [], [], {}
    entries = 0
    for i, layer in enumerate(c.layers):
        ffn = feed_forward_of(layer.mlp)
        block = PreNormBlock(c.width, mixer_of(layer.mixer), ffn, TanhNorm(c.width), TanhNorm(c.width) if ffn else None, BLOCK_NAMES)
        blocks.append(block)
        shared = getattr(layer.mixer, "kv_from", None)
        if shared is None:
            entry_of[i] = entries
            entries += 1
        state = None
        if block.state_need() is not None:
            state = entries
            entries += 1
        schedule.append(LayerRun(i, entry_of[i if shared is None else shared], shared is None, state))
    chain_norms(blocks)
    embedding = TokenEmbedding(c.vocab, c.width, tensor="embed")
    head = OutputHead(c.vocab, c.width, TanhNorm(c.width), tied_to=embedding, norm_name="final.norm")
    return DecoderModel(c, embedding, blocks, head, schedule=schedule, position_encodings=list(rotaries.values()),
                        block_prefix="l{}", embed_prefix="")


register_architecture("Sazisun", SazisunConfig.from_json, build_sazisun)
