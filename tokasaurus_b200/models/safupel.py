"""The Safupel decoder put together from parts, and its registry entry.

A decoder whose blocks read ONE norm (``parts.block.ParallelBlock``: ``x += mixer(N(x)) + ff(N(x))``, an RMS norm whose
weight is stored around zero).  config.json lists the layers one by one; a layer's mixer is a real-gated linear recurrence
behind a short convolution (``parts.recurrent.RealGatedRecurrence``) or chunked attention and matrix memory side by side
(``parts.parallel_mixer.ParallelMixers`` of ``parts.sink_attention.SinkAttention`` with ``chunk`` and ``distance_bias``, and
``parts.recurrent.MatrixMemory``).  Its feed-forward is an ungated exact GELU (``parts.mlp.GeluMLP``), a mixture of
SiLU-gated experts chosen by sigmoid scores that multiply what goes into an expert, with a shared expert
(``parts.mlp.RoutedExperts``), or absent.

Tensor names: ``embed``; per layer i ``l<i>.norm1``, the mixer's ``l<i>.mix.*`` (``.left.*`` / ``.right.*`` of the two sides),
the feed-forward's ``l<i>.mlp.up`` / ``.down`` (dense) or ``.router``, ``.e<j>.gate`` / ``.up`` / ``.down``,
``.shared.gate`` / ``.up`` / ``.down`` (mixture); ``final.norm``; ``head``.
"""

from __future__ import annotations

import torch

from tokasaurus_b200.config.registry import register_architecture
from tokasaurus_b200.config.safupel_config import GatedRecurrenceConfig, SafupelConfig
from tokasaurus_b200.parts import (
    DecoderModel,
    GatedMLP,
    GeluMLP,
    MatrixMemory,
    OutputHead,
    ParallelBlock,
    ParallelMixers,
    RealGatedRecurrence,
    RMSNorm,
    RoutedExperts,
    SinkAttention,
    TokenEmbedding,
)

DECAY_SCALE = 8.0  # the factor in log a = -8 r softplus(lam)
DENOMINATOR_EPS = 1e-6  # added to the matrix memory's denominator
SLOPE_BASE = 8.0  # a head's distance slope is 2^(-8 (h + 1) / heads)


def build_safupel(cfg: SafupelConfig) -> DecoderModel:
    W, eps = cfg.width, cfg.norm_eps
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}", layer.mixer
        if isinstance(m, GatedRecurrenceConfig):
            mixer = RealGatedRecurrence(W, m.width, m.blocks, m.taps, DECAY_SCALE, names=dict(
                y=f"{p}.mix.y", y_b=f"{p}.mix.y.b", x=f"{p}.mix.x", x_b=f"{p}.mix.x.b", conv=f"{p}.mix.conv",
                conv_b=f"{p}.mix.conv.b", ra=f"{p}.mix.ra", ra_b=f"{p}.mix.ra.b", ri=f"{p}.mix.ri", ri_b=f"{p}.mix.ri.b",
                lam=f"{p}.mix.lam", o=f"{p}.mix.o"))
        else:
            a, r = m.left, m.right
            left = SinkAttention(W, a.heads, a.kv_heads, a.dim, a.vdim, a.scale, None, None, eps, q_name=f"{p}.mix.left.q",
                                 k_name=f"{p}.mix.left.k", v_name=f"{p}.mix.left.v", o_name=f"{p}.mix.left.o", sink_name=None,
                                 unit_norm=False, chunk=a.chunk,
                                 distance_bias=[2.0 ** (-SLOPE_BASE * (h + 1) / a.heads) for h in range(a.heads)])
            right = MatrixMemory(W, r.heads, r.dim, r.vdim, r.gate_cap, eps, DENOMINATOR_EPS, names={
                k: f"{p}.mix.right.{t}" for k, t in dict(q="q", k="k", v="v", g="g", o="o", norm="norm", i="i", i_b="i.b",
                                                         f="f", f_b="f.b").items()})
            mixer = ParallelMixers(left, right, m.left_scale, m.right_scale)
        ff = layer.mlp
        if ff is None:
            ffn = None
        elif ff.kind == "dense":
            ffn = GeluMLP(W, ff.ff, f"{p}.mlp.up", f"{p}.mlp.down")
        else:
            shared = None
            if ff.shared_ff is not None:
                shared = GatedMLP(W, ff.shared_ff, f"{p}.mlp.shared.gate", f"{p}.mlp.shared.up", f"{p}.mlp.shared.down",
                                  out_f32=True)
            ffn = RoutedExperts(W, ff.ff, ff.experts, ff.top, f"{p}.mlp.router", None,
                                lambda e, p=p: (f"{p}.mlp.e{e}.gate", f"{p}.mlp.e{e}.up", f"{p}.mlp.e{e}.down"), shared,
                                scored=dict(correction=None, groups=1, keep=1, scale=1.0, renormalize=False),
                                weigh_input=True, out_dtype=torch.float32)
        blocks.append(ParallelBlock(RMSNorm(W, eps, f"{p}.norm1", around_zero=True), mixer, ffn))
    head_norm = RMSNorm(W, eps, "final.norm", around_zero=True, gain=cfg.logit_scale)  # the logits' factor rides in the norm
    return DecoderModel(embedding=TokenEmbedding(cfg.vocab, W, "embed"), blocks=blocks,
                        head=OutputHead(cfg.vocab, W, head_norm, "head"))


register_architecture("Safupel", SafupelConfig.from_dict, build_safupel, model_types=("safupel",), replace=True)
