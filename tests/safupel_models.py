"""Small Safupel models for the tests: configurations whose sizes differ wherever they could be confused, weights with
signs and sizes of their own, and the plain implementation's logits.

Every model exists twice.  ``dyn``: routers whose choice moves from token to token, with margins (asserted here, on the
plain implementation) wide enough that float32 arithmetic cannot turn a choice.  ``tier``: the same model with a stream
whose first channel no sublayer writes and every embedding row starts alike, so that a norm leaves it positive for every
token, and routers that hold one expert a tier on that channel: the choice is then the same for every token while the
chosen experts' scores still move with it.  That is for bfloat16, whose rounding of a router's input would turn close
choices and, through carried states, everything after them."""

from __future__ import annotations

import copy

import numpy as np
import torch

import cuttings
import plain_safupel as plain

F64 = torch.float64


def rec(width, blocks, conv):
    return dict(type="rglru", mixer=dict(width=width, blocks=blocks, conv=conv))


def par(left, right, ls, rs):
    heads, kv, dim, vdim, scale, chunk = left
    a = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale)
    if chunk is not None:
        a["mask"] = dict(size=chunk)
    rh, rd, rv, cap = right
    return dict(type="parallel", mixer=dict(left=a, right=dict(heads=rh, dim=rd, vdim=rv, gate_cap=cap), left_scale=ls, right_scale=rs))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, shared=None):
    d = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared is not None:
        d["shared"] = dict(ff=shared)
    return d


MODELS = {
    # sizes the tensor-core kernels take beside sizes they do not (heads of 24 and 40); parts of 16, 40 and 72 channels;
    # four, three and six taps; chunks that are no multiples of the page size; one, two and all experts chosen, with and
    # without a shared expert; a layer without a feed-forward
    "a": dict(page=8, lengths=[100, 37, 64, 5, 81, 1, 50], seed=12,
              config=dict(architecture="Safupel", vocab=131, width=96, norm=dict(eps=1e-5), logit_scale=1.6,
                          layers=[dict(rec(48, 3, 4), mlp=moe(40, 6, 2, 24)),
                                  dict(par((4, 2, 16, 32, 0.25, 21), (3, 20, 28, 4.0), 1.3, 0.7), mlp=dense(72)),
                                  dict(rec(80, 2, 3), mlp=None),
                                  dict(par((2, 2, 24, 40, 0.2, 37), (2, 16, 16, 9.0), 0.6, 1.1), mlp=moe(32, 4, 1)),
                                  dict(rec(72, 1, 6), mlp=moe(24, 3, 3, 40))])),
    # tensor-core sizes everywhere, experts on the grouped tensor-core path; parts of 128 channels (several column tiles);
    # a chunk of exactly two pages and one of more than a 64-key tile; eight query heads on one key/value head; long requests
    "b": dict(page=16, lengths=[300, 150, 40, 210, 33, 64], seed=12,
              config=dict(architecture="Safupel", vocab=113, width=128, norm=dict(eps=1e-6), logit_scale=0.8,
                          layers=[dict(par((8, 1, 32, 64, 0.18, 32), (4, 32, 64, 6.0), 0.9, 1.2), mlp=moe(64, 8, 4, 64)),
                                  dict(rec(256, 2, 4), mlp=dense(96)),
                                  dict(par((2, 2, 64, 16, 0.125, 100), (1, 64, 48, 15.0), 1.1, 0.5), mlp=moe(72, 3, 1, 40))])),
    # mixers side by side only: no chunks at all, a chunk of one page, three key/value heads of six; one head
    "c": dict(page=8, lengths=[120, 33, 75, 9, 50], seed=11,
              config=dict(architecture="Safupel", vocab=101, width=64, norm=dict(eps=1e-5), logit_scale=1.0,
                          layers=[dict(par((1, 1, 16, 16, 0.3, None), (1, 8, 24, 2.0), 1.0, 1.0), mlp=dense(40)),
                                  dict(par((6, 3, 8, 24, 0.35, 8), (5, 12, 4, 7.0), 0.5, 1.5), mlp=None)])),
    # the recurrence only: no pages at all; one part, parts of one 16-channel tile, a convolution of one tap and of ten
    "d": dict(page=16, lengths=[90, 20, 47, 3, 61], seed=12,
              config=dict(architecture="Safupel", vocab=89, width=80, norm=dict(eps=1e-6), logit_scale=2.5,
                          layers=[dict(rec(64, 4, 2), mlp=moe(32, 5, 2)), dict(rec(96, 1, 1), mlp=dense(48)), dict(rec(40, 5, 10), mlp=dense(56))])),
    # sizes that fit no vector load: a width that is no multiple of four, an odd vocabulary, parts of 13 and 11 channels,
    # odd head sizes and head counts, inner sizes of 26 and 22; two experts of which one is chosen
    "e": dict(page=8, lengths=[70, 21, 44, 2, 33, 17, 26], seed=13,
              config=dict(architecture="Safupel", vocab=77, width=70, norm=dict(eps=1e-5), logit_scale=1.3,
                          layers=[dict(par((3, 1, 10, 13, 0.3, 19), (3, 7, 9, 5.0), 1.4, 0.8), mlp=moe(22, 2, 1, 26)),
                                  dict(rec(39, 3, 4), mlp=dense(26)), dict(rec(22, 2, 3), mlp=None)])),
}

MIN_MARGIN = 5e-5  # of a router's logit: far more than float32 sums of a router's width can move one
TIER_MARGIN = 0.3  # between tiers: far more than bfloat16 rounding of a router's input moves a logit
OUTPUTS = ("mix.o", "mix.left.o", "mix.right.o", "mlp.down")


def adjust(name: str, t: torch.Tensor, g: torch.Generator, tiered: bool) -> torch.Tensor:
    """Vectors get signs and sizes of their own; decays that forget soon and late; see the module's text on ``tiered``."""
    tail = name.split(".", 1)[1] if "." in name else name
    rnd = lambda s: torch.randn(t.shape, generator=g) * s  # noqa: E731
    if name == "embed" or (tail not in OUTPUTS and not tail.endswith(".down")):
        pass
    elif tiered:
        t = t.clone().float()
        t[0] = 0.0  # no sublayer writes the stream's first channel
        return t
    if name == "embed":
        t = t.float() * 6.0
        if tiered:
            t[:, 0] = 9.0
        return t
    if tail in ("norm1", "norm"):
        return rnd(0.25)                                                     # weights around zero
    if tail in ("mix.lam",):
        return torch.linspace(-7.0, 1.5, t.numel())[torch.randperm(t.numel(), generator=g)]
    if tail == "mix.conv":
        return rnd(0.6)
    if tail in ("mix.ra", "mix.ri"):
        return rnd(1.5 / t.shape[-1] ** 0.5)
    if tail == "mix.right.f.b":
        return torch.rand(t.shape, generator=g) * 5.0 + 0.5                  # forgets soon in one head, late in another
    if tail in ("mix.right.i", "mix.right.f"):
        return rnd(0.3)
    if tail == "mix.right.i.b":
        return rnd(1.5)
    if tail.endswith(".b"):
        return rnd(0.4)
    if tail == "mlp.router":
        if not tiered:
            return rnd(0.35)
        E = t.shape[0]
        r = rnd(0.03)
        r[:, 0] = 2.0 * (torch.randperm(E, generator=g).to(torch.float32) - (E - 1.5))
        return r
    return t


def margins(config, w64, tokens):
    """(the smallest gap between the last chosen expert's logit and the first one's that is not, the logits)."""
    zs: list = []
    logits = plain.forward(config, w64, tokens, router_logits=zs)
    gap = float("inf")
    for top, z in zs:
        if top < z.shape[1]:
            s = torch.sort(z, dim=-1, descending=True).values
            gap = min(gap, float((s[:, top - 1] - s[:, top]).min()))
    return gap, logits


def make_models(root, names=None):
    from safetensors import safe_open
    from safetensors.torch import save_file
    from tokasaurus_b200.weights import write_model_folder

    out = {}
    for index, (name, spec) in enumerate(MODELS.items()):
        if names is not None and name not in names:
            continue
        V = spec["config"]["vocab"]
        reqs = {f"{name}{i}": cuttings.random_tokens(n, V, 40 + i) for i, n in enumerate(spec["lengths"])}
        for kind in ("dyn", "tier"):
            folder = write_model_folder(root / f"{name}_{kind}", spec["config"], seed=31 + index, std=0.12, norm_init="uniform")
            w = {}
            with safe_open(str(folder / "model.safetensors"), framework="pt") as f:
                for k in f.keys():
                    w[k] = f.get_tensor(k)
            g = torch.Generator().manual_seed(spec["seed"])
            for k in sorted(w):
                w[k] = adjust(k, w[k], g, kind == "tier").to(w[k].dtype)
            save_file(w, str(folder / "model.safetensors"))
            w64 = {k: v.to(F64) for k, v in w.items()}
            want, noise, margin = {}, {}, float("inf")
            for rid, t in reqs.items():
                mg, logits = margins(spec["config"], w64, t)
                want[rid] = logits.numpy()
                noise[rid] = rounding_noise(spec["config"], w64, t, want[rid], variant_dtype(kind))
                margin = min(margin, mg)
            assert margin > (MIN_MARGIN if kind == "dyn" else TIER_MARGIN), \
                f"model {name} ({kind}): a router's choice rests on a margin of {margin:.2g}"
            out[(name, kind)] = dict(folder=folder, config=spec["config"], weights=w64, reqs=reqs, want=want,
                                     noise=noise, page=spec["page"], margin=margin)
    return out


def variant(dtype: str) -> str:
    return "dyn" if dtype == "float32" else "tier"


def variant_dtype(kind: str) -> str:
    return "float32" if kind == "dyn" else "bfloat16"


def to_bfloat16_and_back(x):
    return x.to(torch.bfloat16).to(x.dtype)


def row_error(d):
    """Per position: the root mean square over the vocabulary of a difference of logits, its mean taken off."""
    return np.sqrt(((d - d.mean(axis=1, keepdims=True)) ** 2).mean(axis=1))


def rounding_noise(config, w64, tokens, want, dtype):
    """How far rounding alone moves the logits at every position: the plain implementation once more, in float32
    arithmetic (``float32``) or in float64 with the operands of the matrix products rounded to bfloat16
    (``bfloat16``), against its float64 logits."""
    if dtype == "float32":
        got = plain.forward(config, w64, tokens, dtype=torch.float32).numpy().astype(np.float64)
    else:
        got = plain.forward(config, w64, tokens, round_fn=to_bfloat16_and_back).numpy()
    return row_error(got - want)


def check_logits(got, m, dtype, what):
    """A position's limit is 3 times what rounding alone does there (``rounding_noise``; at least the request's median,
    since one draw of the rounding can come out small).  No position is over 1.5 times its limit, and at most one in
    fifty (or one) over the limit itself."""
    for rid, ref in m["want"].items():
        noise = m["noise"][rid]
        limit = 3.0 * np.maximum(noise, np.median(noise))
        err = row_error(got[rid] - ref)
        over = np.nonzero(err > limit)[0]
        far = np.nonzero(err > 1.5 * limit)[0]
        assert far.size == 0, (f"{dtype} {what}: request {rid}: first wrong token at position {far[0]} "
                               f"(error {err[far[0]]:.3g}, limit {limit[far[0]]:.3g}); {far.size} of {len(err)} far over")
        assert over.size <= max(1, len(err) // 50), (f"{dtype} {what}: request {rid}: {over.size} of {len(err)} positions "
                                                    f"over their limits, the first at {over[0]}")


def changed(config, path, value):
    """A copy of ``config`` with the entry ``path`` replaced wherever a mixer, a side of it or a feed-forward has it."""
    cfg = copy.deepcopy(config)
    for layer in cfg["layers"]:
        for d in (layer["mixer"], layer.get("mlp")):
            keys = path.split(".")
            while d is not None and len(keys) > 1:
                d = d.get(keys[0])
                keys = keys[1:]
            if d is not None and keys[0] in d:
                d[keys[0]] = value(d[keys[0]])
    return cfg
