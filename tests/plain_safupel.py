"""The Safupel decoder stated plainly: whole sequences, no cache, one function a mechanism, float64 by default.

It shares no code with the engine.  ``forward(cfg, weights, tokens)`` takes the config.json dictionary, a dict of
tensors by name and one sequence's token ids, and returns the logits at every position (and, if asked, the residual
stream after every layer).  ``round_fn`` (identity by default) is applied to the operands of every matrix product that
may run in a lower precision: with a bfloat16 rounding it shows what rounding alone does to the logits.
"""

from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def _ident(x):
    return x


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    """The weight is stored around zero."""
    return rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(u, taps, bias):
    """u [T, C], taps [C, K]: the last column meets the current token, what lies before the first token is zero."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    out = torch.zeros_like(u) + bias
    for k in range(K):
        out = out + taps[:, k] * padded[k:k + T]
    return out


def diagonal_scan(a, x):
    """S_t = a_t * S_(t-1) + x_t from S = 0; a, x [T, C] -> all S_t."""
    s, out = torch.zeros_like(x[0]), []
    for t in range(x.shape[0]):
        s = a[t] * s + x[t]
        out.append(s)
    return torch.stack(out)


def block_product(u, m, bias):
    """u [T, C] in equal parts, m [blocks, n, n] ([out, in] a part), bias [blocks, n] -> [T, C]."""
    B, n, _ = m.shape
    return (torch.einsum("tbi,boi->tbo", u.view(u.shape[0], B, n), m) + bias).reshape(u.shape[0], B * n)


def rglru(h, w, p, m, eps, rnd=_ident):
    """The mixer 'rglru': a diagonal recurrence whose decay and input gate come from the convolved branch."""
    hr = rnd(h)
    y = gelu_tanh(hr @ rnd(w[p + "y"]).T + w[p + "y.b"])
    u = causal_conv(hr @ rnd(w[p + "x"]).T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_product(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_product(u, w[p + "ri"], w[p + "ri.b"]))
    log_a = -8.0 * r * F.softplus(w[p + "lam"])
    s = diagonal_scan(torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u)
    return rnd(s * y) @ rnd(w[p + "o"]).T


def visible(T: int, chunk: int | None):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    ok = j <= i
    if chunk is not None:
        ok = ok & (i // chunk == j // chunk)
    return ok


def slopes(heads: int, dtype=torch.float64):
    return 2.0 ** (-8.0 * (torch.arange(heads, dtype=dtype) + 1.0) / heads)


def distance_attention(q, k, v, scale, mask):
    """q [T, H, d], k [T, H, d], v [T, H, e] -> [T, H, e]; a head's slope times the distance comes off its scores."""
    T, H = q.shape[:2]
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).to(q.dtype)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale - slopes(H, q.dtype)[:, None, None] * dist[None]
    s = s.masked_fill(~mask[None], float("-inf"))
    return torch.einsum("hij,jhe->ihe", torch.softmax(s, dim=-1), v)


def chunked_attention(h, w, p, m, rnd=_ident):
    """Grouped-query attention within chunks of the sequence; up to and without the output projection."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
    hr = rnd(h)
    q = rnd(hr @ rnd(w[p + "q"]).T).view(T, H, d)
    k = rnd(hr @ rnd(w[p + "k"]).T).view(T, G, d).repeat_interleave(H // G, dim=1)
    v = rnd(hr @ rnd(w[p + "v"]).T).view(T, G, e).repeat_interleave(H // G, dim=1)
    o = distance_attention(q, k, v, float(m["scale"]), visible(T, (m.get("mask") or {}).get("size")))
    return o.reshape(T, H * e)


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, d], v [T, H, e], log gates i, f [T, H] -> [T, H, e]: a matrix state and a normaliser a head, scaled by
    a running maximum that starts at 0."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    n = torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        a, c = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = a[:, None, None] * S + c[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + c[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm(h, w, p, m, eps, rnd=_ident):
    """Matrix memory with its gates, head norm and output gate; up to and without the output projection."""
    T = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    hr = rnd(h)
    q = (hr @ rnd(w[p + "q"]).T).view(T, H, d) * d ** -0.5
    k = (hr @ rnd(w[p + "k"]).T).view(T, H, d)
    v = (hr @ rnd(w[p + "v"]).T).view(T, H, e)
    i = soft_cap(hr @ rnd(w[p + "i"]).T + w[p + "i.b"], cap)
    f = F.logsigmoid(soft_cap(hr @ rnd(w[p + "f"]).T + w[p + "f.b"], cap))
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * e) * w[p + "norm"]
    return o * torch.sigmoid(hr @ rnd(w[p + "g"]).T)


def parallel(h, w, p, m, eps, rnd=_ident):
    """The mixer 'parallel': chunked attention and matrix memory side by side."""
    left = rnd(chunked_attention(h, w, p + "left.", m["left"], rnd)) @ rnd(w[p + "left.o"]).T
    right = rnd(mlstm(h, w, p + "right.", m["right"], eps, rnd)) @ rnd(w[p + "right.o"]).T
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


def dense_ff(h, w, p, rnd=_ident):
    return rnd(gelu_erf(rnd(h) @ rnd(w[p + "up"]).T)) @ rnd(w[p + "down"]).T


def expert(h, w, p, rnd=_ident):
    hr = rnd(h)
    return rnd(silu(hr @ rnd(w[p + "gate"]).T) * (hr @ rnd(w[p + "up"]).T)) @ rnd(w[p + "down"]).T


def route(h, w_router, top: int, rnd=_ident):
    """(chosen experts [T, top], their scores [T, top], all logits [T, E])."""
    z = rnd(h) @ w_router.T
    s = torch.sigmoid(z)
    order = torch.sort(z, dim=-1, descending=True, stable=True).indices[:, :top]
    return order, torch.gather(s, 1, order), z


def moe_ff(h, w, p, mlp, rnd=_ident):
    """A chosen expert's score multiplies what goes IN."""
    r = mlp["router"]
    idx, wt, _ = route(h, w[p + "router"], int(r["top"]), rnd)
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        rows, slot = (idx == e).nonzero(as_tuple=True)
        if rows.numel():
            out[rows] += expert(h[rows] * wt[rows, slot][:, None], w, f"{p}e{e}.", rnd)
    if mlp.get("shared"):
        out = out + expert(h, w, p + "shared.", rnd)
    return out


MIXERS = {"rglru": rglru, "parallel": parallel}


def forward(cfg: dict, w: dict, tokens, dtype=torch.float64, round_fn=None, layers_out: list | None = None,
            router_logits: list | None = None):
    rnd = round_fn or _ident
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        up = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, rnd)
        mlp = layer.get("mlp")
        if mlp is not None:
            up = up + (dense_ff(h, w, p + "mlp.", rnd) if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp, rnd))
            if router_logits is not None and mlp["kind"] == "moe":
                router_logits.append((int(mlp["router"]["top"]), route(h, w[p + "mlp.router"], 1, rnd)[2]))
        x = x + up
        if layers_out is not None:
            layers_out.append(x.clone())
    return rnd(rms_norm(x, w["final.norm"], eps)) @ rnd(w["head"]).T * float(cfg["logit_scale"])
