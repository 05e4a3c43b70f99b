"""The Deletar decoder put together from parts, and its registry entry.

A decoder with a norm ahead of every sublayer and another on its output (``parts.block.SandwichNormBlock``, RMS norms whose
weights are stored around zero), over a scaled embedding, with capped logits.  config.json lists the layers one by one.
All three mixers are windowed grouped-query attention with a rotation in halves on part of a head
(``parts.sink_attention.SinkAttention``):

* "attention": a short convolution on every channel of q, k and v behind their projections;
* "attention_2": biases, values that are the keys as projected, q and k normed over the whole projection, capped scores, an
  output gate a head;
* "attention_3": q and k normed a head, rotation frequencies scaled by wavelength, capped scores, a one in the softmax's
  denominator, an output gate a head.

A layer may read the keys and values that an earlier layer cached.  The feed-forward is the square of relu without a gate
(``parts.mlp.SquaredReluMLP``), a mixture of such experts that a table of token ids chooses, with a shared expert
(``parts.mlp.RoutedExperts`` with ``table_name``), or absent.

Tensor names: ``embed``; per layer i ``l<i>.norm1`` / ``.norm1b`` / ``.norm2`` / ``.norm2b``, the mixer's ``l<i>.mix.*``, the
feed-forward's ``l<i>.mlp.up`` / ``.down`` (dense) or ``.table``, ``.e<j>.up`` / ``.down``, ``.shared.up`` / ``.down``
(mixture); ``final.norm``; ``head``.
"""

from __future__ import annotations

import torch

from tokasaurus_b200.config.deletar_config import DeletarConfig
from tokasaurus_b200.config.registry import register_architecture
from tokasaurus_b200.parts import (
    DecoderModel,
    LayerCall,
    OutputHead,
    RMSNorm,
    RotaryEncoding,
    RoutedExperts,
    SandwichNormBlock,
    SinkAttention,
    SquaredReluMLP,
    TokenEmbedding,
)


def _rotary(rot):
    if rot is None:
        return None
    if rot.scaling is None:
        return RotaryEncoding(rot.dims, rot.base)
    s = rot.scaling
    return RotaryEncoding(rot.dims, rot.base, "llama3", factor=s.factor, low_freq_factor=s.low, high_freq_factor=s.high,
                          original_max_position_embeddings=s.original)


def kept_windows(cfg: DeletarConfig) -> dict[int, int | None]:
    """How many positions each layer's cached keys must stay for, the layers that read them included (None: all)."""
    keep: dict[int, int | None] = {}
    for i, layer in enumerate(cfg.layers):
        src, w = (i if layer.mixer.kv_from is None else layer.mixer.kv_from), layer.mixer.window
        keep[src] = w if src not in keep else (None if w is None or keep[src] is None else max(keep[src], w))
    return keep


def build_deletar(cfg: DeletarConfig) -> DecoderModel:
    W, eps = cfg.width, cfg.norm_eps
    keep = kept_windows(cfg)
    blocks, order = [], []
    for i, layer in enumerate(cfg.layers):
        p, m, kind = f"l{i}", layer.mixer, layer.type
        q, k, v = f"{p}.mix.q", f"{p}.mix.k", f"{p}.mix.v"
        own = m.kv_from is None
        src = i if own else m.kv_from
        options: dict = dict(own_kv=own, cache_window=keep[src], rotary=_rotary(m.rot), rotary_pairs=False)
        if kind == "attention":
            options.update(unit_norm=False, conv=(m.taps, (f"{q}.conv", f"{k}.conv", f"{v}.conv")))
        else:
            options.update(unit_norm=True, qk_norm_names=(f"{q}.norm", f"{k}.norm"), gate_name=f"{p}.mix.g")
            if kind == "attention_2":
                options.update(values_are_keys=True, bias_names=(f"{q}.b", f"{k}.b", ""), norm_over="projection")
            else:
                options.update(null_sink=True)
        mixer = SinkAttention(W, m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.softcap, m.window, eps, q_name=q, k_name=k,
                              v_name=None if kind == "attention_2" else v, o_name=f"{p}.mix.o", sink_name=None, **options)
        ff = layer.mlp
        ffn = None
        if ff is not None and ff.kind == "dense":
            ffn = SquaredReluMLP(W, ff.ff, f"{p}.mlp.up", f"{p}.mlp.down")
        elif ff is not None:
            shared = None
            if ff.shared_ff is not None:
                shared = SquaredReluMLP(W, ff.shared_ff, f"{p}.mlp.shared.up", f"{p}.mlp.shared.down")
            ffn = RoutedExperts(W, ff.ff, ff.experts, ff.top, None, None,
                                lambda e, p=p: (f"{p}.mlp.e{e}.up", f"{p}.mlp.e{e}.down"), shared, expert="relu2",
                                out_dtype=torch.float32, table_name=f"{p}.mlp.table", vocab=cfg.vocab)

        def norm(name):
            return RMSNorm(W, eps, f"{p}.{name}", around_zero=True)

        if ffn is None:
            blocks.append(SandwichNormBlock(norm("norm1"), mixer, norm("norm1b")))
        else:
            blocks.append(SandwichNormBlock(norm("norm1"), mixer, norm("norm1b"), norm("norm2"), ffn, norm("norm2b")))
        order.append(LayerCall(i, src, write_cache=own))
    return DecoderModel(
        embedding=TokenEmbedding(cfg.vocab, W, "embed", scale=cfg.embedding_scale), blocks=blocks,
        head=OutputHead(cfg.vocab, W, RMSNorm(W, eps, "final.norm", around_zero=True), "head", softcap=cfg.logit_softcap),
        run_order=order)


register_architecture("Deletar", DeletarConfig.from_dict, build_deletar, model_types=("deletar",), replace=True)
