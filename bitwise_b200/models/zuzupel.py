"""Zuzupel assembled from parts, and its entry in the architecture registry.

A decoder whose layers carry a layer norm (a weight, no bias) on each sublayer's output only: ``x += norm1(mixer(x))``,
``x += norm2(ff(x))`` (``PostNormBlock``).  Three kinds of mixer, in any order:

* ``wkv``: a recurrence whose projections each read a mix of the current and the previous row, with a decay from the
  input and a bonus for the current token (``ShiftedRecurrence``);
* ``channel_delta``: the gated delta rule with a decay per key channel and a short convolution on q, k and v
  (``ChannelDelta``);
* ``parallel``: attention inside chunks (biased projections, weighted norms per head, a rotation in the half layout with
  frequencies divided by a factor) and a matrix memory side by side (``PairedMixer``).

The feed-forward is ``W_down relu(W_up h)^2`` or absent.  A layer may run another layer's block with a cache or state of
its own.  The head has weights of its own behind a last layer norm.

Tensor names: ``embed``, ``final.norm``, ``head``, and per layer ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*`` (see
the mixers), ``l<i>.mlp.{up, down}``.  Matrices are stored [out, in].
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zuzupel import ZuzupelConfig
from ..parts.block import PostNormBlock
from ..parts.embedding import OutputHead, TokenEmbedding
from ..parts.mlp import DenseFFN
from ..parts.norm import LayerNorm
from ..parts.paired import PairedMixer
from ..parts.rope import HalfRotaryEncoding, LinearScaling
from ..parts.scored_attention import ScoredAttention
from ..parts.state_recurrence import ChannelDelta, MatrixMemory, ShiftedRecurrence
from .decoder import DecoderModel, LayerRun

BLOCK_NAMES = {"mixer": "mix", "mixer_post": "norm1", "feed_forward": "mlp", "ffn_post": "norm2"}


def build_zuzupel(config: ZuzupelConfig) -> DecoderModel:
    c = config

    def norm():
        return LayerNorm(c.width, c.eps, suffix="")

    rotaries = {}   # one table per (turned entries, base, factor)

    def mixer_of(m):
        if m.kind == "wkv":
            return ShiftedRecurrence(c.width, m.heads, m.dim, m.decay_rank or max(1, m.dim // 2), c.eps)
        if m.kind == "channel_delta":
            return ChannelDelta(c.width, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, m.decay_rank or max(1, m.dim // 2),
                                m.gate_rank or max(1, m.dim // 2), c.eps)
        a, r = m.left, m.right
        rotary = None
        if a.rot_dims:
            key = (a.rot_dims, a.rot_base, a.rot_factor)
            if key not in rotaries:
                rotaries[key] = HalfRotaryEncoding(a.rot_dims, a.rot_base, LinearScaling(a.rot_factor) if a.rot_factor else None)
            rotary = rotaries[key]
        left = ScoredAttention(c.width, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, c.eps, qk_norm=True, position=rotary,
                               rot_dims=a.rot_dims or 0, bias=True, chunk=a.chunk)
        return PairedMixer(c.width, left, MatrixMemory(c.width, r.heads, r.dim, r.vdim, r.gate_cap, c.eps), c.eps)

    blocks, prefixes, schedule, block_of = [], [], [], {}
    entries = 0
    for i, layer in enumerate(c.layers):
        j = c.owner(i)
        if j not in block_of:
            block_of[j] = len(blocks)
            ffn = DenseFFN(c.width, layer.ff) if layer.ff else None
            blocks.append(PostNormBlock(c.width, mixer_of(c.layers[j].mixer), ffn, norm(), norm() if ffn else None, BLOCK_NAMES,
                                        opens=i == 0))
            prefixes.append(f"l{j}")
        block = blocks[block_of[j]]
        cache_entry, state_entry = entries, None
        entries += 1
        if block.state_need() is not None:
            state_entry = entries
            entries += 1
        schedule.append(LayerRun(block_of[j], cache_entry, True, state_entry))
    embedding = TokenEmbedding(c.vocab, c.width, tensor="embed")
    head = OutputHead(c.vocab, c.width, norm(), norm_name="final.norm", head_name="head", suffix="")
    return DecoderModel(c, embedding, blocks, head, schedule=schedule, position_encodings=list(rotaries.values()),
                        embed_prefix="", block_prefixes=prefixes)


register_architecture("Zuzupel", ZuzupelConfig.from_json, build_zuzupel)
