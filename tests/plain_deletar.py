"""The Deletar decoder stated plainly: whole sequences, no cache, one function a mechanism, float64 by default.

It shares no code with the engine.  ``forward(cfg, weights, tokens)`` takes the config.json dictionary, a dict of
tensors by name and one sequence's token ids, and returns the logits at every position (and, if asked, the residual
stream after every layer).  ``round_fn`` (identity by default) is applied to the operands of every matrix product that
may run in a lower precision: with a bfloat16 rounding it shows what rounding alone does to the logits.
"""

from __future__ import annotations

import math

import torch


def _ident(x):
    return x


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    """The weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def causal_conv(u, taps):
    """u [T, C], taps [C, K]: the last column meets the current token, what lies before the first token is zero."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    out = torch.zeros_like(u)
    for k in range(K):
        out = out + taps[:, k] * padded[k:k + T]
    return out


def frequencies(rot):
    """A pair's angle per position, float64 [dims / 2]; with ``scaling``, low frequencies are divided by a factor, high ones
    are kept, and those between are a blend (by wavelength, against the length they were trained on)."""
    n, base = int(rot["dims"]), float(rot["base"])
    out = []
    sc = rot.get("scaling")
    for i in range(n // 2):
        f = base ** (-2.0 * i / n)
        if sc is not None:
            factor, low, high, orig = (float(sc[k]) for k in ("factor", "low", "high", "original"))
            wave = 2.0 * math.pi / f
            if wave > orig / low:
                f = f / factor
            elif not wave < orig / high:
                s = (orig / wave - low) / (high - low)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_half(x, freq):
    """x [T, heads, d]: channel i turns with channel i + n, i below n = len(freq); the channels from 2n on stay."""
    T, n = x.shape[0], freq.shape[0]
    a = torch.arange(T, dtype=torch.float64)[:, None, None] * freq
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def visible(T: int, window: int | None):
    """Position i sees itself and the window - 1 positions before it."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    ok = d >= 0
    return ok if window is None else ok & (d < window)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def softmax_attention(q, k, v, scale, mask, cap=None, null_key=False):
    """q [T, H, d], k [T, H, d], v [T, H, e] -> [T, H, e].  ``null_key``: a key of score 0 and value 0 takes part."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    if cap is not None:
        s = soft_cap(s, cap)
    s = s.masked_fill(~mask[None], float("-inf"))
    if null_key:
        s = torch.cat([s, torch.zeros_like(s[..., :1])], dim=-1)
    p = torch.softmax(s, dim=-1)
    if null_key:
        p = p[..., :-1]
    return torch.einsum("hij,jhe->ihe", p, v)


def _sizes(m):
    H = int(m["heads"])
    return H, int(m.get("kv_heads", H)), int(m["dim"]), int(m["vdim"])


def _turn(x, m):
    return rotate_half(x, frequencies(m["rot"])) if m.get("rot") else x


def _window(m):
    return (m.get("mask") or {}).get("size")


def keys_values(h, w, p, m, kind, eps, rnd=_ident):
    """What a layer caches: keys [T, G, d] after norm and rotation, values [T, G, e]."""
    T = h.shape[0]
    _, G, d, e = _sizes(m)
    hr = rnd(h)
    k = hr @ rnd(w[p + "k"]).T
    if kind == "attention":
        k = causal_conv(k, w[p + "k.conv"])
        v = causal_conv(hr @ rnd(w[p + "v"]).T, w[p + "v.conv"])
        k = k.view(T, G, d)
    elif kind == "attention_2":
        k = k + w[p + "k.b"]
        v = k  # as projected
        k = (rms(k, eps) * w[p + "k.norm"]).view(T, G, d)  # one norm over all heads' channels
    else:
        v = hr @ rnd(w[p + "v"]).T
        k = rms(k.view(T, G, d), eps) * w[p + "k.norm"]
    return rnd(_turn(k, m)), rnd(v.view(T, G, e))


def queries(h, w, p, m, kind, eps, rnd=_ident):
    T = h.shape[0]
    H, _, d, _ = _sizes(m)
    q = rnd(h) @ rnd(w[p + "q"]).T
    if kind == "attention":
        q = causal_conv(q, w[p + "q.conv"]).view(T, H, d)
    elif kind == "attention_2":
        q = (rms(q + w[p + "q.b"], eps) * w[p + "q.norm"]).view(T, H, d)
    else:
        q = rms(q.view(T, H, d), eps) * w[p + "q.norm"]
    return rnd(_turn(q, m))


def attention(h, w, p, m, kind, eps, kv, rnd=_ident):
    """One of the three mixers, given the keys and values that it reads."""
    T = h.shape[0]
    H, G, d, e = _sizes(m)
    q = queries(h, w, p, m, kind, eps, rnd)
    k, v = (t.repeat_interleave(H // G, dim=1) for t in kv)
    cap = None if kind == "attention" else float(m["softcap"])
    o = softmax_attention(q, k, v, float(m["scale"]), visible(T, _window(m)), cap, null_key=kind == "attention_3")
    if kind != "attention":
        o = o * torch.sigmoid(rnd(h) @ rnd(w[p + "g"]).T)[:, :, None]
    return rnd(o.reshape(T, H * e)) @ rnd(w[p + "o"]).T


def squared_relu_ff(h, w, p, rnd=_ident):
    return rnd(torch.relu(rnd(h) @ rnd(w[p + "up"]).T) ** 2) @ rnd(w[p + "down"]).T


def table_moe(h, w, p, mlp, tokens, rnd=_ident):
    """A table gives each token id its experts, which count alike."""
    table = w[p + "table"].long()[torch.as_tensor(tokens, dtype=torch.long)]
    top = int(mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(int(mlp["router"]["experts"])):
        rows = (table == e).any(-1).nonzero()[:, 0]
        if rows.numel():
            out[rows] += squared_relu_ff(h[rows], w, f"{p}e{e}.", rnd) / top
    if mlp.get("shared"):
        out = out + squared_relu_ff(h, w, p + "shared.", rnd)
    return out


def forward(cfg: dict, w: dict, tokens, dtype=torch.float64, round_fn=None, layers_out: list | None = None):
    rnd = round_fn or _ident
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.", layer["mixer"], layer["type"]
        h = rms_norm(x, w[p + "norm1"], eps)
        src = m.get("kv_from")
        cached[i] = keys_values(h, w, p + "mix.", m, kind, eps, rnd) if src is None else cached[src]
        x = x + rms_norm(attention(h, w, p + "mix.", m, kind, eps, cached[i], rnd), w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            y = (squared_relu_ff(h, w, p + "mlp.", rnd) if mlp["kind"] == "dense"
                 else table_moe(h, w, p + "mlp.", mlp, tokens, rnd))
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = rnd(rms_norm(x, w["final.norm"], eps)) @ rnd(w["head"]).T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else soft_cap(logits, float(cap))
