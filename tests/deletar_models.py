"""Small Deletar models for the tests: configurations whose sizes differ wherever they could be confused, weights with
signs and sizes of their own, and the plain implementation's logits.  (No choice in this design rests on rounding: one set
of weights a model serves both precisions.)"""

from __future__ import annotations

import copy

import numpy as np
import torch

import cuttings
import plain_deletar as plain

F64 = torch.float64


def layer(kind, heads, kv_heads, dim, vdim, window, rot, mlp, conv=None, softcap=None, scale=None, kv_from=None):
    """``rot``: (dims, base) or (dims, base, factor, low, high, original)."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale if scale is not None else 1.3 * dim ** -0.5,
             rot=dict(dims=rot[0], base=rot[1]))
    if len(rot) > 2:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), rot[2:]))
    for key, v in (("conv", conv), ("softcap", softcap), ("kv_from", kv_from)):
        if v is not None:
            m[key] = v
    if window is not None:
        m["mask"] = dict(size=window)
    return dict(type=kind, mixer=m, mlp=mlp)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, shared=None):
    d = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))
    if shared is not None:
        d["shared"] = dict(ff=shared)
    return d


def model(vocab, width, eps, scale, softcap, layers):
    d = dict(architecture="Deletar", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)
    if softcap is not None:
        d["logit_softcap"] = softcap
    return d


A, A2, A3 = "attention", "attention_2", "attention_3"
MODELS = {
    # sizes the tensor-core kernels take beside sizes they do not (keys of 24, values of 40); two and four taps; windows that
    # are no multiples of the page size; a layer that reads another's rows with more heads and a wider window of its own; one
    # layer without a window; one, two and all experts chosen, with and without a shared expert; a layer without a feed-forward
    "a": dict(page=8, lengths=[100, 37, 64, 5, 81, 1, 50], seed=21, config=model(131, 96, 1e-5, 1.7, 12.0, [
        layer(A, 4, 2, 16, 32, 21, (8, 5000.0), dense(72), conv=4),
        layer(A2, 6, 2, 24, 24, 13, (24, 10000.0), moe(40, 6, 2, 24), softcap=8.0),
        layer(A3, 4, 4, 32, 48, 37, (20, 800.0, 6.0, 1.0, 3.0, 90), None, softcap=5.0),
        layer(A3, 8, 4, 32, 48, 50, (20, 800.0, 6.0, 1.0, 3.0, 90), moe(32, 4, 1), softcap=3.0, kv_from=2, scale=0.3),
        layer(A, 3, 1, 24, 40, None, (10, 300.0), moe(24, 3, 3, 40), conv=2)])),
    # tensor-core sizes everywhere, experts on the grouped tensor-core path; windows of exactly two pages, of one 64-key tile
    # and of more; twenty query heads on one key/value head; a reader whose window is narrower than its source's; long requests
    "b": dict(page=16, lengths=[300, 150, 40, 210, 33, 64], seed=22, config=model(113, 128, 1e-6, 3.0, 20.0, [
        layer(A3, 20, 1, 32, 64, 100, (16, 9000.0, 4.0, 1.0, 4.0, 64), moe(64, 8, 4, 64), softcap=6.0),
        layer(A2, 2, 2, 64, 64, 64, (32, 700.0), dense(96), softcap=4.0),
        layer(A, 8, 4, 32, 16, 32, (32, 250000.0), moe(72, 3, 1, 40), conv=3),
        layer(A3, 4, 1, 32, 64, 70, (16, 9000.0, 4.0, 1.0, 4.0, 64), dense(64), softcap=9.0, kv_from=0)])),
    # a window of one token and of one page, one tap, two readers of one layer (one before and one behind another mixer, the
    # wider window last), one head, rotation of the whole head; logits without a cap; the last layer reads another's rows
    "c": dict(page=8, lengths=[120, 33, 75, 9, 50], seed=23, config=model(101, 64, 1e-5, 0.6, None, [
        layer(A, 1, 1, 16, 16, 1, (16, 100.0), dense(40), conv=1),
        layer(A3, 6, 3, 8, 24, 8, (8, 50.0, 3.0, 1.0, 2.0, 30), None, softcap=2.0),
        layer(A3, 3, 3, 8, 24, 3, (8, 50.0, 3.0, 1.0, 2.0, 30), moe(16, 2, 1), softcap=7.0, kv_from=1),
        layer(A2, 4, 1, 16, 16, 19, (4, 60.0), moe(40, 5, 2), softcap=6.0),
        layer(A3, 6, 3, 8, 24, 26, (8, 50.0, 3.0, 1.0, 2.0, 30), dense(24), softcap=4.0, kv_from=1)])),
    # the other two mixers as readers of another layer's rows; two convolutions of the same rows' shape; six taps
    "d": dict(page=16, lengths=[90, 20, 47, 3, 61], seed=24, config=model(89, 80, 1e-6, 2.0, 7.0, [
        layer(A, 4, 2, 16, 16, 25, (12, 400.0), dense(48), conv=6),
        layer(A, 6, 2, 16, 16, 40, (12, 400.0), moe(32, 5, 2, 16), conv=3, kv_from=0),
        layer(A2, 2, 1, 32, 32, 17, (16, 90.0), dense(40), softcap=3.0),
        layer(A2, 3, 1, 32, 32, 17, (16, 90.0), None, softcap=5.0, kv_from=2)])),
    # sizes that fit no vector load: a width that is no multiple of four, an odd vocabulary, odd head sizes and counts, inner
    # sizes of 26 and 22; two experts of which one is chosen
    "e": dict(page=8, lengths=[70, 21, 44, 2, 33, 17, 26], seed=25, config=model(77, 70, 1e-5, 1.3, 9.0, [
        layer(A, 3, 1, 10, 13, 19, (6, 200.0), moe(22, 2, 1, 26), conv=5),
        layer(A2, 3, 3, 9, 9, 11, (2, 30.0), dense(26), softcap=4.0),
        layer(A3, 5, 1, 14, 7, 30, (14, 70.0, 5.0, 0.5, 2.5, 40), moe(22, 7, 3), softcap=3.0)])),
}


def adjust(name: str, t: torch.Tensor, g: torch.Generator) -> torch.Tensor:
    """Vectors get signs and sizes of their own."""
    tail = name.split(".", 1)[1] if "." in name else name
    rnd = lambda s: torch.randn(t.shape, generator=g) * s  # noqa: E731
    if tail in ("norm1", "norm1b", "norm2", "norm2b", "norm"):
        return rnd(0.25)                                             # weights around zero
    if tail in ("mix.q.norm", "mix.k.norm"):
        return (torch.rand(t.shape, generator=g) + 0.7) * torch.randn(t.shape, generator=g).sign()
    if tail.endswith(".conv"):
        return rnd(0.6)
    if tail.endswith(".b"):
        return rnd(0.4)
    if tail == "mix.g":
        return rnd(1.5 / t.shape[1] ** 0.5)
    if name == "embed":
        return t.float() * 5.0
    return t


def make_models(root, names=None):
    from safetensors import safe_open
    from safetensors.torch import save_file
    from tokasaurus_b200.weights import write_model_folder

    out = {}
    for index, (name, spec) in enumerate(MODELS.items()):
        if names is not None and name not in names:
            continue
        V = spec["config"]["vocab"]
        reqs = {f"{name}{i}": cuttings.random_tokens(n, V, 60 + i) for i, n in enumerate(spec["lengths"])}
        folder = write_model_folder(root / name, spec["config"], seed=51 + index, std=0.12, norm_init="uniform")
        w = {}
        with safe_open(str(folder / "model.safetensors"), framework="pt") as f:
            for k in f.keys():
                w[k] = f.get_tensor(k)
        g = torch.Generator().manual_seed(spec["seed"])
        for k in sorted(w):
            w[k] = adjust(k, w[k], g).to(w[k].dtype)
        save_file(w, str(folder / "model.safetensors"))
        w64 = {k: v.to(F64) if v.is_floating_point() else v for k, v in w.items()}
        want = {rid: plain.forward(spec["config"], w64, t).numpy() for rid, t in reqs.items()}
        noise = {dt: {rid: rounding_noise(spec["config"], w64, t, want[rid], dt) for rid, t in reqs.items()}
                 for dt in ("float32", "bfloat16")}
        out[name] = dict(folder=folder, config=spec["config"], weights=w64, reqs=reqs, want=want, noise=noise, page=spec["page"])
    return out


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


def check_logits(got, want, noise, dtype, what):
    """A position's limit is 3 times what rounding alone does there (``rounding_noise``; at least the request's median,
    since one draw of the rounding can come out small).  No position is over 1.5 times its limit, and at most one in
    fifty (or one) over the limit itself."""
    for rid, ref in want.items():
        limit = 3.0 * np.maximum(noise[rid], np.median(noise[rid]))
        err = row_error(got[rid] - ref)
        over = np.nonzero(err > limit)[0]
        far = np.nonzero(err > 1.5 * limit)[0]
        assert far.size == 0, (f"{dtype} {what}: request {rid}: first wrong token at position {far[0]} "
                               f"(error {err[far[0]]:.3g}, limit {limit[far[0]]:.3g}); {far.size} of {len(err)} far over")
        assert over.size <= max(1, len(err) // 50), (f"{dtype} {what}: request {rid}: {over.size} of {len(err)} positions "
                                                    f"over their limits, the first at {over[0]}")


def changed(config, path, value):
    """A copy of ``config`` with the entry ``path`` replaced wherever a mixer or a feed-forward has it."""
    cfg = copy.deepcopy(config)
    for ly in cfg["layers"]:
        for d in (ly["mixer"], ly.get("mlp")):
            keys = path.split(".")
            while d is not None and len(keys) > 1:
                d = d.get(keys[0])
                keys = keys[1:]
            if d is not None and keys[0] in d:
                d[keys[0]] = value(d[keys[0]])
    return cfg
