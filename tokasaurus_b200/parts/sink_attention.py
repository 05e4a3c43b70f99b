"""Grouped-query attention over a sliding window with a cap on the scores and a sink in the softmax.

q = W_q h + b_q, k = W_k h + b_k (``dim`` values a head), v = W_v h + b_v (``vdim`` values a head; the two sizes may
differ); optionally every q head and every k head is divided by its root mean square (an RMS norm without a weight);
no rotation.  With c the cap,

    s_ij = c * tanh(scale * q_i . k_j / c),      o_i = sum_j exp(s_ij) v_j / (exp(sink_h) + sum_j exp(s_ij))

over the last ``window`` positions (the query's own included; None: all).  The sink is a learned number per head that
takes part in the denominator only.  The output projection may carry a bias (``out_bias``), which the block adds.

A token's key and value of one key/value head are cached side by side as one row [k | v] (one plane): rows
``[page, kv head, slot, dim + vdim]``.  The projections are one product with a float32 result; biases, the unit norms,
scores, weights and sums are float32.  In float32, and for head sizes that are no multiples of 16, one FP32-pipe kernel
serves every token; in bfloat16 otherwise the tensor-core kernels of csrc/attention_sink.cu do (weights rounded to
bfloat16 for their product with the values, as in the framework's other attention kernels).

Options that other designs bring: a weight vector on the q and k norms (``qk_norm_names``); a rotation of q and k by
position on the first ``rotary.rotary_dim`` channels of a head, in neighbouring pairs or in halves (``rotary``,
``rotary_pairs``; after the norm); values that ARE the keys as projected, before norm and rotation
(``values_are_keys``: no W_v, vdim = dim); a learned factor on every head's scale and a learned number added to its
scores (``head_scale_name``, ``head_bias_name``); and ``weights="sigmoid"``: no softmax, the weight of a visible key
is sigmoid(score), not normalised over the keys (then there is no sink).

``keep_first``: with a window, a request's first so many positions stay visible to every later query (position i sees
j if j <= i and (i - j < window or j < keep_first)); their pages stay in the cache.  ``maps`` > 1: so many attention
maps a head, each with query and key vectors of its own (q and k hold them head by head, [map 0 | map 1 | ...]) and a
softmax of its own over the same values; the cached row is [k of map 0 | k of map 1 | ... | v].  What becomes of the
maps' outputs is a subclass's business (``_combine``; ``parts.diff_attention.DifferentialAttention``).  ``extra_names``:
further matrices over the mixer's input whose rows ride in the same product as q, k and v (an output gate's, say);
their float32 results are the trailing columns of the product that ``_combine`` is handed.

``chunk``: instead of a sliding window, the sequence is cut into chunks of so many positions, counted from position 0,
and a query sees the keys of its own chunk only; pages of earlier chunks go back.  ``distance_bias``: a number a head;
that slope times the distance i - j comes off the scores, after scale and cap.

``conv``: a short causal convolution over time on every channel of q, k and v, directly behind the projections
(``parts.conv`` adds one to a norm's rows; this one stands alone): y_t = sum_j w[:, j] * u_(t - n + 1 + j) with n taps and
zeros before the first token.  A request's last n - 1 projected rows are its state, float32, a side entry of the mixer.
``norm_over="projection"``: q, and k, are each divided by ONE root mean square over all their heads; the weights then have
the projections' sizes.  ``null_sink``: every head's sink has the score 0 (a one in the denominator), without a tensor.
``gate_name``: head h's result is multiplied by sigmoid(W_g x)_h before the output projection; the gate's matrix rides in
the q|k|v product and the attention kernels apply it to the unrounded result.
``own_kv=False``: the layer has no keys and values of its own; it reads the rows that another layer's call has cached
(``cache_window``: how many positions that entry keeps, at least this mixer's window), with its own queries and mask.

A mixer that stands beside others reads a share of ONE input product and leaves its rows for ONE output product:
``in_matrix`` / ``out_matrix`` are the matrices it wants there, ``mix`` is what lies between them.
"""

from __future__ import annotations

import torch

from tokasaurus_b200.kernels import ops
from tokasaurus_b200.parts.base import Mixer, PagedCacheNeed, StateNeed, WeightSpec


class SinkAttention(Mixer):
    graph_safe = True

    def __init__(self, width: int, n_heads: int, n_kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: float | None, window: int | None, norm_eps: float, q_name: str, k_name: str, v_name: str,
                 o_name: str, sink_name: str | None, bias_names: tuple[str, str, str] | None = None,
                 out_bias_name: str | None = None, unit_norm: bool = True, qk_norm_names: tuple[str, str] | None = None,
                 rotary=None, rotary_pairs: bool = True, values_are_keys: bool = False,
                 head_scale_name: str | None = None, head_bias_name: str | None = None, weights: str = "softmax",
                 keep_first: int = 0, maps: int = 1, extra_names: tuple[tuple[str, int], ...] = (),
                 chunk: int | None = None, distance_bias=None, conv: tuple[int, tuple[str, str, str]] | None = None,
                 norm_over: str = "head", null_sink: bool = False, gate_name: str | None = None, own_kv: bool = True,
                 cache_window: int | None | str = "same"):
        """``extra_names``: (tensor name, rows) of matrices [rows, width] appended to the q|k|v product.  ``conv``: (taps, the tensor
        names of q's, k's and v's taps [channels, taps])."""
        if n_heads % n_kv_heads:
            raise ValueError(f"n_heads={n_heads} is not a multiple of n_kv_heads={n_kv_heads}")
        if weights not in ("softmax", "sigmoid"):
            raise ValueError(f"attention weights are 'softmax' or 'sigmoid', not {weights!r}")
        if weights == "sigmoid" and sink_name is not None:
            raise ValueError("sigmoid weights are not normalised: there is no sink")
        if values_are_keys and vdim != dim:
            raise ValueError(f"values that are the keys have the keys' size {dim}, not {vdim}")
        if qk_norm_names is not None and not unit_norm:
            raise ValueError("norm weights need the norm")
        if maps < 1 or (maps > 1 and (values_are_keys or type(self) is SinkAttention)):
            raise ValueError("several attention maps a head need a part that combines them, and values of their own")
        if keep_first < 0 or (keep_first and not window):
            raise ValueError("positions kept in sight need a window to be kept from")
        if chunk and window:
            raise ValueError("a chunk or a sliding window, not both")
        if distance_bias is not None and (len(distance_bias) != n_heads or maps != 1):
            raise ValueError(f"{len(distance_bias)} distance slopes for {n_heads} heads of {maps} maps")
        if norm_over not in ("head", "projection"):
            raise ValueError(f"a norm of q and k is over a 'head' or the 'projection', not {norm_over!r}")
        if norm_over == "projection" and (not unit_norm or qk_norm_names is None):
            raise ValueError("a norm over the projection comes with its weights")
        if conv is not None and (conv[0] < 1 or bias_names is not None or values_are_keys or norm_over == "projection"):
            raise ValueError("a convolution has at least one tap; with biases, values that are the keys, or a norm over the "
                             "projection it is not built")
        if null_sink and (sink_name is not None or weights == "sigmoid"):
            raise ValueError("a sink of score 0 takes the place of a learned one, in a softmax")
        if gate_name is not None and maps != 1:
            raise ValueError("an output gate within the attention needs one map a head")
        if gate_name is not None:
            extra_names = tuple(extra_names) + ((gate_name, n_heads),)
        self.gated, self.null_sink, self.own_kv = gate_name is not None, bool(null_sink), bool(own_kv)
        self.whole_norm = norm_over == "projection"
        self.taps, self.conv_names = (int(conv[0]), tuple(conv[1])) if conv is not None else (0, None)
        self.conv_w: torch.Tensor | None = None
        if chunk and cache_window != "same":
            raise ValueError("a chunk's keys are kept as long as the chunk")
        if cache_window != "same" and cache_window is not None and (not window or window > cache_window):
            raise ValueError(f"a window of {window} positions cannot be read from a cache entry that keeps {cache_window}")
        self.cache_window = cache_window
        self.chunk = int(chunk) if chunk else None
        self.distance_bias = tuple(float(x) for x in distance_bias) if distance_bias is not None else None
        self.head_slope: torch.Tensor | None = None
        self.maps, self.keep_first, self.extra_names = int(maps), int(keep_first), tuple(extra_names)
        if rotary is not None and rotary.rotary_dim > dim:
            raise ValueError(f"{rotary.rotary_dim} rotated channels in heads of {dim}")
        self.sigmoid = weights == "sigmoid"
        self.qk_norm_names, self.rotary, self.rotary_pairs = qk_norm_names, rotary, bool(rotary_pairs)
        self.values_are_keys = bool(values_are_keys)
        self.head_scale_name, self.head_bias_name = head_scale_name, head_bias_name
        self.qk_norm_w = self.rot_freq = self.head_scale = self.head_bias = None
        self.width, self.n_heads, self.n_kv_heads, self.dim, self.vdim = width, n_heads, n_kv_heads, dim, vdim
        self.scale = float(scale)
        self.softcap = float(softcap) if softcap else None
        self.window = int(window) if window else None
        self.norm_eps, self.unit_norm = float(norm_eps), bool(unit_norm)
        self.names = (q_name, k_name, v_name, o_name)
        self.sink_name, self.bias_names, self.out_bias_name = sink_name, bias_names, out_bias_name
        self.defines = ops.sink_attention_defines(dim, vdim, self.sigmoid, self.maps, self.distance_bias is not None, self.taps)
        self.sinks = self.qkv_bias = self.out_bias = None

    def weight_specs(self):
        q, k, v, o = self.names
        H, G, d, e = self.n_heads, self.n_kv_heads, self.dim, self.vdim
        M = self.maps
        own = self.own_kv
        specs = [WeightSpec(q, (H * M * d, self.width))]
        if own:
            specs.append(WeightSpec(k, (G * M * d, self.width)))
        specs.append(WeightSpec(o, (self.width, H * e)))
        specs += [WeightSpec(n, (rows, self.width)) for n, rows in self.extra_names]
        if own and not self.values_are_keys:
            specs.append(WeightSpec(v, (G * e, self.width)))
        if self.qk_norm_names is not None:
            sizes = (H * M * d, G * M * d) if self.whole_norm else (d, d)
            specs += [WeightSpec(n, (c,), role="vector") for n, c in list(zip(self.qk_norm_names, sizes))[:2 if own else 1]]
        if self.conv_names is not None:
            specs += [WeightSpec(n, (c, self.taps), role="vector")
                      for n, c in list(zip(self.conv_names, (H * M * d, G * M * d, G * e)))[:3 if own else 1]]
        specs += [WeightSpec(n, (H * M,), role="vector") for n in (self.head_scale_name, self.head_bias_name) if n is not None]
        if self.bias_names is not None:
            specs += [WeightSpec(n, (rows,), role="vector")
                      for n, rows in zip(self._own_biases(), (H * M * d, G * M * d, G * e))]
        if self.out_bias_name is not None:
            specs.append(WeightSpec(self.out_bias_name, (self.width,), role="vector"))
        if self.sink_name is not None:
            specs.append(WeightSpec(self.sink_name, (H * M,), role="vector"))
        return tuple(specs)

    def _own_biases(self):
        """The names of the biases on what the mixer projects itself."""
        return self.bias_names[:(2 if self.values_are_keys else 3) if self.own_kv else 1]

    def kernel_modules(self, dtype):
        return (("attention_sink.cu", self.defines),)

    def _conv_columns(self) -> int:
        H, G, M = self.n_heads, self.n_kv_heads, self.maps
        return H * M * self.dim + (G * (M * self.dim + self.vdim) if self.own_kv else 0)

    def side_needs(self):
        if self.taps < 2:
            return {}
        return {"conv": StateNeed(((self.taps - 1) * self._conv_columns(),), "float32")}

    def cache_need(self):
        window = self.window if self.cache_window == "same" else self.cache_window
        return PagedCacheNeed(self.n_kv_heads, self.maps * self.dim + self.vdim, self.chunk or window, planes=1,
                              keep_first=self.keep_first, chunked=self.chunk is not None)

    def bind(self, weights, rt) -> None:
        q, k, v, o = self.names
        stack = [weights[q]]
        if self.own_kv:
            stack += [weights[k]] + ([] if self.values_are_keys else [weights[v]])
        # where the extra matrices' results start in a row of the product
        self.extra_off = sum(w.shape[0] for w in stack)
        stack += [weights[n] for n, _ in self.extra_names]
        self.gate_off = sum(w.shape[0] for w in stack) - self.n_heads  # (the gate's matrix is the last)
        odd = -sum(w.shape[0] for w in stack) % 8
        if self.gated and odd:  # the product's rows stay whole 16-byte pieces
            stack.append(torch.zeros((odd, self.width), dtype=stack[0].dtype, device=stack[0].device))
        self.w_qkv = torch.cat(stack, dim=0).contiguous()
        self.w_o = weights[o].contiguous()
        if self.bias_names is not None:
            self.qkv_bias = torch.cat([weights[n].float() for n in self._own_biases()]).contiguous()
        if self.qk_norm_names is not None:
            # (a mixer without keys of its own: the second weight is never read)
            names = self.qk_norm_names if self.own_kv else self.qk_norm_names[:1] * (1 if self.whole_norm else 2)
            join = torch.cat if self.whole_norm else torch.stack
            self.qk_norm_w = join([weights[n].float() for n in names]).contiguous()
        if self.conv_names is not None:
            self.conv_w = torch.cat([weights[n].float() for n in self.conv_names[:3 if self.own_kv else 1]], dim=0).contiguous()
        if self.rotary is not None and self.rotary.rotary_dim > 0:
            self.rot_freq = self.rotary.inv_freq64().to(rt.device)
        if self.distance_bias is not None:
            self.head_slope = torch.tensor(self.distance_bias, dtype=torch.float64).float().to(rt.device)
        if self.head_scale_name is not None:
            self.head_scale = weights[self.head_scale_name].contiguous()
        if self.head_bias_name is not None:
            self.head_bias = weights[self.head_bias_name].contiguous()
        if self.out_bias_name is not None:
            self.out_bias = weights[self.out_bias_name].contiguous()
        if self.sink_name is not None:
            self.sinks = weights[self.sink_name].contiguous()
        elif self.null_sink:
            self.sinks = torch.zeros((self.n_heads * self.maps,), dtype=torch.float32, device=rt.device)

    def _combine(self, ctx, attn, qkv, out_rows):
        """What goes into the output projection, from the attention's result ``attn`` ([rows, heads * maps * vdim]; with
        several maps float32) and the float32 product ``qkv`` of all tokens; ``out_rows`` names the tokens of attn's
        rows (None: all)."""
        return attn

    def in_matrix(self) -> torch.Tensor:
        return self.w_qkv

    def out_matrix(self) -> torch.Tensor:
        return self.w_o

    def drop_matrices(self) -> None:
        """The matrices live on in a wider product."""
        self.w_qkv = self.w_o = None

    def forward(self, ctx, h, cache, out_rows=None, side=None):
        qkv = ops.linear(h, self.w_qkv, out_dtype=torch.float32)
        return ops.linear_out_f32(self.mix(ctx, qkv, cache, h.dtype, out_rows, side=side), self.w_o, ctx.status)

    def mix(self, ctx, qkv, cache, dtype, out_rows=None, out=None, out_scale: float = 1.0, side=None):
        """From the float32 product ``qkv`` of all tokens (a column slice will do) to what the output product reads, times
        ``out_scale``, in ``dtype``.  ``out`` (one map, all rows): where it goes, a column slice of a wider tensor."""
        H, G, d, e, M = self.n_heads, self.n_kv_heads, self.dim, self.vdim, self.maps
        T, dev = qkv.shape[0], qkv.device
        tables = ctx.tables[cache.group]
        q = torch.empty((T, H * M * d), dtype=dtype, device=dev)
        prep = dict(norm_w=self.qk_norm_w, rot_freq=self.rot_freq, rot_pairs=self.rotary_pairs,
                    rot_dims=self.rotary.rotary_dim if self.rot_freq is not None else 0, maps=M, own_kv=self.own_kv,
                    sigmoid=self.sigmoid, distance=self.head_slope is not None)
        if self.taps:
            state = side["conv"] if self.taps > 1 else None
            ops.sink_attn_conv_prep(qkv, self.conv_w, state.state if state is not None else None, self.unit_norm,
                                    self.norm_eps, q, cache.k, ctx.positions, ctx.token_seq, ctx.seq_slot, ctx.seq_q_start,
                                    ctx.seq_q_len, ctx.n_seqs, not ctx.single_token_step, tables.indptr, tables.page_ids, H, G,
                                    d, e, cache.page_size, cache.writable, state is not None and state.writable, ctx.status,
                                    **prep)
        else:
            ops.sink_attn_prep(qkv, self.qkv_bias, self.unit_norm, self.norm_eps, q, cache.k, ctx.positions, ctx.token_seq,
                               tables.indptr, tables.page_ids, H, G, d, e, cache.page_size, cache.writable, ctx.status,
                               values_are_keys=self.values_are_keys, whole_norm=self.whole_norm, **prep)
        out_dtype = dtype if M == 1 else torch.float32  # several maps' outputs stay unrounded for what combines them
        options = dict(head_scale=self.head_scale, head_bias=self.head_bias, sigmoid=self.sigmoid, maps=M,
                       keep_first=self.keep_first, chunk=self.chunk, head_slope=self.head_slope, out_scale=out_scale,
                       gate=qkv[:, self.gate_off:self.gate_off + H] if self.gated else None, taps=self.taps)
        if ops.can_use_attn_sink_tc(dtype, d, e, M):
            # bfloat16: every token on the tensor cores (single tokens and portions by a kernel each); wanted rows are
            # cut out afterwards
            attn = out if out is not None else torch.empty((T, H * M * e), dtype=out_dtype, device=dev)
            ops.attn_sink_tc(q, attn, cache.k, ctx.seq_q_start, ctx.seq_q_len, ctx.seq_kv_len, tables.indptr,
                             tables.page_ids, ctx.n_seqs, self.sinks, H, G, d, e, cache.page_size, self.scale, self.softcap,
                             self.window, ctx.status, portions=not ctx.single_token_step, **options)
            if out_rows is not None:
                cut = torch.empty((out_rows.numel(), H * M * e), dtype=out_dtype, device=dev)
                ops.gather_rows(attn, out_rows, cut)
                attn = cut
            return self._combine(ctx, attn, qkv, out_rows)
        n_rows = T if out_rows is None else out_rows.numel()
        attn = out if out is not None else torch.empty((n_rows, H * M * e), dtype=out_dtype, device=dev)
        ops.attn_sink(q, attn, cache.k, ctx.token_seq, ctx.positions, tables.indptr, tables.page_ids, out_rows, n_rows,
                      self.sinks, H, G, d, e, cache.page_size, self.scale, self.softcap, self.window, ctx.status, **options)
        return self._combine(ctx, attn, qkv, out_rows)
