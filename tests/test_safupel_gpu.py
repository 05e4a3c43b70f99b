"""The Safupel decoder on the GPU against the plain implementation in ``plain_safupel`` (float64, whole sequences, no
cache): every mechanism's kernels alone, then small random models of several shapes (``safupel_models``) through trace
replay in four cuttings and both precisions with pools that hold exactly what a trace needs, the stream layer by
layer, long decoding, and greedy generation through the engine's entry point and scheduler."""

import numpy as np
import pytest
import torch

import cuttings
import plain_safupel as plain
import safupel_models as sm

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def rel_err(got, want):
    want = np.asarray(want, dtype=np.float64)
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / max(np.abs(want).max(), 1e-30))


def row_err(got, want):
    """The largest error of a row relative to that row's largest value."""
    want = np.asarray(want, dtype=np.float64)
    d = np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=1)
    return float((d / np.maximum(np.abs(want).max(axis=1), 1e-30)).max())


@pytest.fixture(scope="module")
def ops():
    from tokasaurus_b200.kernels import ops as o
    return o


def paged(n_tokens, page, seed):
    """A block table of scattered pages for one request."""
    n_pages = -(-n_tokens // page)
    perm = np.random.default_rng(seed).permutation(n_pages + 5)[:n_pages]
    return [int(p) for p in perm], n_pages + 5


def step_tables(pieces):
    """The request tables of a step whose request r brings pieces[r] tokens: (token_seq, seq_q_start, seq_q_len)."""
    starts = [0] + [int(x) for x in np.cumsum(pieces)][:-1]
    return i32([r for r, n in enumerate(pieces) for _ in range(n)]), i32(starts), i32(list(pieces))


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,H", [(1, 96), (5, 70), (16, 2048), (130, 384), (3, 33)])
def test_norm_adds_two_updates_and_counts_its_weight_from_one(ops, dtype, rows, H):
    """The norm of a block whose sublayers stand side by side: a pair of float32 updates, each rows or K-split slices; the
    weight stored around zero, times a gain."""
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import ResidualStream, RMSNorm

    g = torch.Generator().manual_seed(rows + H)
    w = torch.randn(H, generator=g) * 0.3
    norm = RMSNorm(H, 1e-5, "n", around_zero=True, gain=1.7)
    norm.bind({"n": w.to(DEV)}, Runtime.make(DEV, dtype))
    for s1, s2 in ((3, 5), (1, 4), (0, 1), (0, 0), (4, None), (0, None)):
        def update(s):
            return torch.randn((s, rows, H) if s else (rows, H), generator=g)
        x, a = torch.randn(rows, H, generator=g), update(s1)
        b = update(s2) if s2 is not None else None
        total = x.double() + (a.double().sum(0) if s1 else a.double())
        if b is not None:
            total = total + (b.double().sum(0) if s2 else b.double())
        stream = ResidualStream(x.to(DEV), a.to(DEV) if b is None else (a.to(DEV), b.to(DEV)))
        out = norm.forward(None, stream)
        assert stream.delta is None and rel_err(stream.x.cpu(), total) < 1e-6
        assert rel_err(out.float().cpu(), plain.rms_norm(total, w.double(), 1e-5) * 1.7) < (2e-6 if dtype == "float32" else 6e-3)


def chunked_case(raw, heads, kv, dim, vdim, scale, chunk):
    """Attention from raw projections [n, q | k | v] with plain's building blocks."""
    n = raw.shape[0]
    q = raw[:, :heads * dim].double().view(n, heads, dim)
    k = raw[:, heads * dim:(heads + kv) * dim].double().view(n, kv, dim).repeat_interleave(heads // kv, dim=1)
    v = raw[:, (heads + kv) * dim:(heads + kv) * dim + kv * vdim].double().view(n, kv, vdim).repeat_interleave(heads // kv, dim=1)
    return plain.distance_attention(q, k, v, scale, plain.visible(n, chunk)).reshape(n, heads * vdim)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim,page,heads,kv,chunk", [
    (16, 32, 16, 4, 2, 37), (32, 64, 16, 8, 1, 64), (24, 40, 8, 2, 2, 50), (64, 16, 16, 2, 2, 16), (48, 80, 16, 20, 1, 130),
    (10, 13, 8, 3, 3, 40), (32, 32, 16, 2, 1, None), (128, 128, 16, 4, 2, 100)])
def test_attention_within_chunks_and_with_a_distance_bias(ops, dtype, dim, vdim, page, heads, kv, chunk):
    """Made-up keys that made-up queries score far above all others stand (a) at a chunk's first position, asked for by the
    chunk's last query (just inside, as far away as can be), and (b) at a chunk's last position, asked for by the next
    chunk's first query (just outside, one token away); without chunks, far away.  In one piece, in portions (cut in the
    middle of a chunk and right at its edge) and token by token, on the FP32 pipes and (in bfloat16, for sizes they take)
    on the tensor cores beside a second request of one token.  The result is a share of wider rows, times a factor."""
    n, factor = 330, 0.7
    g = torch.Generator().manual_seed(dim + page + heads)
    C = (heads + kv) * dim + kv * vdim
    scale = dim ** -0.5
    raw = torch.randn(n, C + 5, generator=g)
    u = torch.randn(dim, generator=g).sign() * (30.0 / dim ** 0.5) ** 0.5  # aligned pairs score 30 / dim^0.5 * dim * scale
    size = chunk or 160
    inside, outside = (size, 2 * size - 1), (3 * size - 1, 3 * size)
    if outside[1] >= n:
        outside = (size - 1, size)
    for key, query in (inside, outside):
        raw[key, heads * dim:(heads + kv) * dim] = u.repeat(kv)
        raw[query, :heads * dim] = u.repeat(heads)
    raw = raw.to(torch.bfloat16).float() if dtype == "bfloat16" else raw
    want = chunked_case(raw, heads, kv, dim, vdim, scale, chunk) * factor
    if chunk is not None:  # the plain result at these queries rests on the chunks' edges
        for other, row in ((chunk - 1, inside[1]), (None, outside[1])):
            moved = chunked_case(raw, heads, kv, dim, vdim, scale, other) * factor
            assert float((moved[row] - want[row]).abs().max()) > 0.1 * float(want[row].abs().max())
    slope = plain.slopes(heads).float().to(DEV)
    table, n_pages = paged(n, page, 7)
    single_raw = torch.randn(1, C + 5, generator=g).to(torch.bfloat16).float()
    stable, spages = [0], 1
    tol = 2e-5 if dtype == "float32" else 2e-2
    for cut in ([n], [size + 1, 3, 2, 1], [size, size // 2 + 1, 2]):
        cut = cut + [min(64, n - sum(cut))] + [1] * 3 if sum(cut) < n else [n]
        cut += [n - sum(cut)] if sum(cut) < n else []
        for tc in ([False, True] if ops.can_use_attn_sink_tc(DT[dtype], dim, vdim) else [False]):
            cache = torch.full((n_pages + spages, kv, page, dim + vdim), float("nan"), dtype=DT[dtype], device=DEV)
            status = torch.zeros(1, dtype=torch.int32, device=DEV)
            at, outs = 0, []
            for m in cut:
                beside = tc  # a second request with one token at position 0
                rows = torch.cat([raw[at:at + m], single_raw]) if beside else raw[at:at + m]
                T = m + (1 if beside else 0)
                seq, q_start, q_len = step_tables([m, 1] if beside else [m])
                pos = i32(list(range(at, at + m)) + ([0] if beside else []))
                tabs = [table[:-(-(at + m) // page)]] + ([[n_pages + stable[0]]] if beside else [])
                indptr, ids = i32([0] + [int(x) for x in np.cumsum([len(t) for t in tabs])]), i32([p for t in tabs for p in t])
                q = torch.empty(T, heads * dim, dtype=DT[dtype], device=DEV)
                rd = rows.to(DEV)
                ops.sink_attn_prep(rd, None, False, 1e-6, q, cache, pos, seq, indptr, ids, heads, kv, dim, vdim, page, True, status,
                                   distance=True)
                wide = torch.full((T, heads * vdim + 8), 9.0, dtype=DT[dtype], device=DEV)
                out = wide[:, 4:4 + heads * vdim] if not tc or (4 * 2) % 8 == 0 else wide[:, :heads * vdim]
                kw = dict(chunk=chunk, head_slope=slope, out_scale=factor)
                if tc:
                    kv_len = i32([at + m, 1])
                    ops.attn_sink_tc(q, out, cache, q_start, q_len, kv_len, indptr, ids, 2, None, heads, kv, dim, vdim, page, scale,
                                     None, None, status, **kw)
                else:
                    ops.attn_sink(q, out, cache, seq, pos, indptr, ids, None, T, None, heads, kv, dim, vdim, page, scale, None, None,
                                  status, **kw)
                assert bool((wide[:, :4] == 9.0).all()) and bool((wide[:, 4 + heads * vdim:] == 9.0).all())
                outs.append(out[:m].float().cpu())
                if beside:
                    alone = chunked_case(single_raw, heads, kv, dim, vdim, scale, chunk) * factor
                    assert rel_err(out[m:].float().cpu(), alone) < tol
                at += m
            assert int(status.item()) == 0
            assert row_err(torch.cat(outs), want) < tol, (tc, cut)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,d,e,cap", [(4, 48, 48, 12.0), (3, 7, 9, 5.0), (2, 128, 128, 15.0), (1, 64, 20, 3.0), (5, 33, 130, 8.0)])
def test_matrix_memory_in_portions_and_beside_others(ops, dtype, H, d, e, cap):
    """Gates, walk with its column of ones, and head norm, as the part between its products: one request of 700 tokens in
    portions (longer than a round of the gates' scan, down to two and one token), others beside it, a slot taken over from
    a request that ended.  A token far back writes with an input gate that nothing after it comes near, and is asked for
    at the end; the carried state (float32 whatever the engine's precision) matches the plain one."""
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import MatrixMemory

    eps, den_eps, width = 1e-6, 1e-6, 16
    names = {k: k for k in ("q", "k", "v", "g", "o", "norm", "i", "i_b", "f", "f_b")}
    part = MatrixMemory(width, H, d, e, cap, eps, den_eps, names)
    g = torch.Generator().manual_seed(H * d + e)
    i_b, f_b = torch.randn(H, generator=g), torch.rand(H, generator=g) * 4 + 1.0
    norm_w = torch.rand(H * e, generator=g) + 0.5
    C = 2 * H * d + 2 * H * e + 2 * H
    weights = {n: torch.zeros(s.shape) for n in names.values() for s in part.weight_specs() if s.name == n}
    weights.update(i_b=i_b, f_b=f_b, norm=norm_w)
    part.bind({k: v.to(DEV) for k, v in weights.items()}, Runtime.make(DEV, dtype))

    def request(n, seed, strong_at=None):
        p = torch.randn(n, C, generator=torch.Generator().manual_seed(seed))
        p[:, -2 * H:] *= 2.0
        if strong_at is not None:
            p[strong_at, -2 * H:-H] += 4 * cap
            p[n - 1, :H * d] = p[strong_at, H * d:2 * H * d] * 3  # the last query asks for that key
        return p

    def want(p):
        n, x = p.shape[0], p.double()
        o = 2 * H * d
        q, k = x[:, :H * d].view(n, H, d) * d ** -0.5, x[:, H * d:o].view(n, H, d)
        v, gate = x[:, o:o + H * e].view(n, H, e), x[:, o + H * e:o + 2 * H * e]
        i = plain.soft_cap(x[:, o + 2 * H * e:o + 2 * H * e + H] + i_b.double(), cap)
        f = torch.nn.functional.logsigmoid(plain.soft_cap(x[:, -H:] + f_b.double(), cap))
        out = plain.rms(plain.matrix_memory(q, k, v, i, f), eps).reshape(n, H * e) * norm_w.double()
        return out * torch.sigmoid(gate)

    reqs = {"a": request(700, 1, 5), "b": request(41, 2, 3), "c": request(9, 3), "d": request(64, 4, 0)}
    plan = [{"a": 600, "b": 3}, {"a": 2, "b": 1, "c": 1}, {"c": 8, "b": 30}, {"a": 1, "b": 7}, {"a": 1, "d": 33}, {"a": 96, "d": 1}, {"d": 30}]
    slots = {"a": 2, "b": 0, "c": 1, "d": 0}  # d takes over b's slot
    state = torch.zeros((4, part.cache_need().shape[0]), dtype=torch.float32, device=DEV)
    at, outs = dict.fromkeys(reqs, 0), {r: [] for r in reqs}

    class Ctx:
        pass

    class Cache:
        writable = True
    Cache.state = state
    for step in plan:
        for r in step:
            if at[r] == 0:
                state[slots[r]].zero_()
        ctx = Ctx()
        _, ctx.seq_q_start, ctx.seq_q_len = step_tables(list(step.values()))
        ctx.seq_slot, ctx.n_seqs = i32([slots[r] for r in step]), len(step)
        rows = torch.cat([reqs[r][at[r]:at[r] + n] for r, n in step.items()])
        # the product's rows are wider than this part's share, and so are the rows it writes
        proj = torch.cat([torch.randn(rows.shape[0], 8, generator=g), rows], dim=1).to(DEV)[:, 8:]
        wide = torch.full((rows.shape[0], H * e + 16), 9.0, dtype=DT[dtype], device=DEV)
        part.mix(ctx, proj, Cache, DT[dtype], out=wide[:, 8:8 + H * e], out_scale=0.6)
        assert bool((wide[:, :8] == 9.0).all()) and bool((wide[:, 8 + H * e:] == 9.0).all())
        lo = 0
        for r, n in step.items():
            outs[r].append(wide[lo:lo + n, 8:8 + H * e].float().cpu())
            at[r] += n
            lo += n
    for r, p in reqs.items():
        ref = want(p) * 0.6
        got = torch.cat(outs[r])
        # a head's output is divided by its own size: rows are compared with the size of all rows
        assert rel_err(got, ref) < (2e-4 if dtype == "float32" else 8e-3), r
        assert float((((got.double() - ref) ** 2).mean() / (ref ** 2).mean()).sqrt()) < (2e-5 if dtype == "float32" else 4e-3), r


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,parts,K", [(128, 2, 4), (39, 3, 4), (80, 2, 3), (22, 2, 3), (256, 1, 4), (96, 8, 1), (600, 2, 10), (72, 1, 6)])
def test_real_gated_recurrence_in_portions_and_beside_others(ops, dtype, C, parts, K):
    """Convolution, gates, scan and output branch between the products: portions that end and begin inside the tiles of
    the scan, requests side by side within a tile, steps of single tokens, a slot taken over.  Decays from about 1 - 1e-4
    to 0.  The carried state is float32 whatever the engine's precision and matches the plain one to float32 accuracy (the
    gates' matrices are bfloat16 numbers, their inputs are not rounded)."""
    n_part = C // parts
    g = torch.Generator().manual_seed(C + K)
    rnd = lambda *s: torch.randn(*s, generator=g)  # noqa: E731
    y_b, x_b, taps, conv_b = rnd(C) * 0.5, rnd(C) * 0.5, rnd(C, K) * 0.6, rnd(C) * 0.3
    ra, ri = (rnd(parts, n_part, n_part) * (1.5 / n_part ** 0.5)).bfloat16(), (rnd(parts, n_part, n_part) * (1.5 / n_part ** 0.5)).bfloat16()
    ra_b, ri_b = rnd(C), rnd(C)
    lam = torch.linspace(-11.0, 2.0, C)[torch.randperm(C, generator=g)]
    neg = (-8.0 * torch.nn.functional.softplus(lam.double())).float()

    def request(n, seed):
        return torch.randn(n, 2 * C, generator=torch.Generator().manual_seed(seed))

    def want(p):
        y = plain.gelu_tanh(p[:, :C].double() + y_b.double())
        u = plain.causal_conv(p[:, C:].double() + x_b.double(), taps.double(), conv_b.double())
        r = torch.sigmoid(plain.block_product(u, ra.double(), ra_b.double().view(parts, -1)))
        i = torch.sigmoid(plain.block_product(u, ri.double(), ri_b.double().view(parts, -1)))
        log_a = r * neg.double()
        s = plain.diagonal_scan(torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a)) * i * u)
        return s, s * y

    reqs = {"a": request(500, 1), "b": request(90, 2), "c": request(9, 3), "d": request(61, 4), "e": request(1, 5)}
    plan = [{"a": 300, "b": 3}, {"a": 2, "b": 1, "c": 1, "e": 1}, {"c": 5, "b": 70, "a": 1}, {"a": 1, "b": 1, "c": 1}, {"b": 15, "c": 2},
            {"a": 130, "d": 40}, {"d": 2, "a": 2}, {"d": 1, "a": 1}, {"a": 63, "d": 18}]
    slots = {"a": 2, "b": 0, "c": 1, "d": 0, "e": 3}
    state = torch.full((5, C * K), float("nan"), dtype=torch.float32, device=DEV)
    dev = lambda t: t.to(DEV).contiguous()  # noqa: E731
    vec = [dev(t) for t in (y_b, x_b, taps, conv_b)]
    mats = [dev(ra.to(DT[dtype])), dev(ra_b), dev(ri.to(DT[dtype])), dev(ri_b)]
    at, outs = dict.fromkeys(reqs, 0), {r: [] for r in reqs}
    for step in plan:
        for r in step:
            if at[r] == 0:
                state[slots[r]].zero_()
        seq, q_start, q_len = step_tables(list(step.values()))
        rows = torch.cat([reqs[r][at[r]:at[r] + n] for r, n in step.items()])
        pad = 2 if rows.shape[0] < 50 else 0  # padding tokens, as a step graph has them
        proj = torch.cat([rows, torch.full((pad, 2 * C), float("nan"))]).to(DEV)
        out = torch.empty((rows.shape[0] + pad, C), dtype=DT[dtype], device=DEV)
        ops.real_gated_recurrence(proj, 0, C, *vec, *mats, dev(neg), state, torch.cat([seq, i32([-1] * pad)]),
                                  i32([slots[r] for r in step]), q_start, q_len, out)
        lo = 0
        for r, n in step.items():
            outs[r].append(out[lo:lo + n].float().cpu())
            at[r] += n
            lo += n
            s = want(reqs[r][:at[r]])[0][-1]
            assert rel_err(state[slots[r], :C].cpu(), s) < 1e-5, (r, at[r])
            kept = torch.cat([torch.zeros(K, C), reqs[r][:at[r], C:] + x_b])[-(K - 1):] if K > 1 else torch.zeros(0, C)
            assert torch.equal(state[slots[r], C:].cpu().view(K - 1, C), kept.float()) if K > 1 and at[r] >= K - 1 else True
    for r, p in reqs.items():
        assert at[r] == p.shape[0]
        assert rel_err(torch.cat(outs[r]), want(p)[1]) < (1e-5 if dtype == "float32" else 5e-3), r
    assert bool(torch.isnan(state[4]).all())  # nobody's slot


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,inner", [(1, 64, 40), (7, 96, 72), (16, 70, 26), (40, 128, 96), (200, 96, 136), (130, 70, 26)])
def test_ungated_feed_forward_with_the_exact_gelu(ops, dtype, T, H, inner):
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import GeluMLP

    g = torch.Generator().manual_seed(T + inner)
    w = {"up": (torch.randn(inner, H, generator=g) * 0.25).bfloat16(), "down": (torch.randn(H, inner, generator=g) * 0.2).bfloat16()}
    h = torch.randn(T, H, generator=g).to(DT[dtype])
    part = GeluMLP(H, inner, "up", "down")
    part.bind({k: v.to(DEV, DT[dtype]) for k, v in w.items()}, Runtime.make(DEV, dtype))
    got = part.forward(None, h.to(DEV))
    assert got.dtype == torch.float32
    got = (got.sum(0) if got.dim() == 3 else got).cpu()
    assert rel_err(got, plain.dense_ff(h.double(), {k: v.double() for k, v in w.items()}, "")) < (1e-5 if dtype == "float32" else 1.5e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,top,H,inner,shared", [(3, 4, 2, 64, 40, 24), (5, 6, 1, 96, 32, None), (70, 8, 4, 128, 64, 64),
                                                    (400, 5, 5, 96, 72, 40), (150, 3, 2, 128, 64, None), (33, 2, 1, 70, 22, 26),
                                                    (700, 4, 1, 70, 22, None)])
def test_experts_whose_scores_weigh_their_input(ops, dtype, T, E, top, H, inner, shared):
    """The routed feed-forward as a part: the largest sigmoid scores, not renormalised, multiply what goes into the experts
    (few rows, tiled, and in bfloat16 the grouped tensor-core products), beside a shared expert."""
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import GatedMLP, RoutedExperts

    g = torch.Generator().manual_seed(T + E)
    w = {"router": torch.randn(E, H, generator=g) * 0.2}
    for e in list(range(E)) + (["s"] if shared else []):
        p, n = (f"e{e}", inner) if e != "s" else ("shared", shared)
        w[p + ".gate"], w[p + ".up"] = torch.randn(n, H, generator=g) * 0.25, torch.randn(n, H, generator=g) * 0.25
        w[p + ".down"] = torch.randn(H, n, generator=g) * 0.25
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    mlp = dict(kind="moe", expert=dict(ff=inner), router=dict(experts=E, top=top), shared=dict(ff=shared) if shared else None)
    h = torch.randn(T, H, generator=g).to(DT[dtype])
    sh = GatedMLP(H, shared, "shared.gate", "shared.up", "shared.down", out_f32=True) if shared else None
    part = RoutedExperts(H, inner, E, top, "router", None, lambda e: (f"e{e}.gate", f"e{e}.up", f"e{e}.down"), sh,
                         scored=dict(renormalize=False), weigh_input=True, out_dtype=torch.float32)
    part.bind({k: v.to(DEV) if k == "router" else v.to(DEV, DT[dtype]) for k, v in w.items()}, Runtime.make(DEV, dtype))
    got = part.forward(None, h.to(DEV)).cpu()
    w64 = {k: v.double() for k, v in w.items()}
    z = torch.sort(h.double() @ w64["router"].T, dim=-1, descending=True).values
    assert top == E or float((z[:, top - 1] - z[:, top]).min()) > 1e-5  # no choice rests on a close call
    want = plain.moe_ff(h.double(), w64, "", mlp)
    assert got.dtype == torch.float32 and rel_err(got, want) < (3e-5 if dtype == "float32" else 2e-2)
    # weighing the outputs instead is another function
    idx, wt, _ = plain.route(h.double(), w64["router"], top)
    other = torch.stack([sum(wt[t, j] * plain.expert(h[t:t + 1].double(), w64, f"e{int(idx[t, j])}.")[0] for j in range(top)) for t in range(min(T, 8))])
    if shared:
        other = other + plain.expert(h[:8].double(), w64, "shared.")
    assert rel_err(other, want[:8]) > 0.05


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return sm.make_models(tmp_path_factory.mktemp("safupel_models"))


CUTS = dict(whole=cuttings.whole, prefix_then_single=cuttings.prefix_then_single,
            changing_portions=cuttings.changing_portions, mixed=cuttings.mixed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("which", list(sm.MODELS))
def test_cuttings_match_plain(models, which, cut, dtype):
    """Whole prompts, prompts then single tokens, portions of changing size down to one and two tokens, and up to four
    requests side by side in four slots, in a pool that holds exactly what the trace needs: pages and slots are used again
    (pages of earlier chunks within a request's own life, too), and a later request must see nothing of an earlier one's
    keys and states."""
    from tokasaurus_b200.engine.trace import TraceReplayer

    m = models[(which, sm.variant(dtype))]
    steps = CUTS[cut](m["reqs"])
    rp = TraceReplayer(str(m["folder"]), dtype, cuttings.max_live_tokens(steps, m["page"]), page_size=m["page"], max_requests=4)
    cache = rp.runner.cache
    owners, users, outs = {}, {}, []
    for st in steps:
        outs.append(rp.run_step(st))
        cache.check()
        for rid, rc in cache.requests.items():
            users.setdefault(rc.slot, set()).add(rid)
            for gi in range(len(cache.groups)):
                for p in rc.live_pages(gi):
                    owners.setdefault((gi, p), set()).add(rid)
                first = cache.groups[gi].need.first_visible(rp.lengths[rid]) // m["page"]
                assert all((p < 0) == (i < first) for i, p in enumerate(rc.tables[gi])), "pages before the chunk go back, others stay"
    assert not cache.requests and cache.num_free_pages() == [g.allocator.num_pages for g in cache.groups]
    sm.check_logits(cuttings.collect(steps, outs), m, dtype, cut)
    if cut == "mixed":
        assert any(len(v) > 1 for v in users.values()), "no slot was used by two requests"
        assert not cache.groups or any(len(v) > 1 for v in owners.values()), "no page was used by two requests"


def test_layer_by_layer(models):
    """The residual stream after every layer, float32, one prompt in one step and in two."""
    from tokasaurus_b200.engine.batch import StepEntry
    from tokasaurus_b200.engine.trace import TraceReplayer

    for which in sm.MODELS:
        m = models[(which, "dyn")]
        rid, toks = next(iter(m["reqs"].items()))
        want = []
        plain.forward(m["config"], m["weights"], toks, layers_out=want)
        for cut in ([len(toks)], [len(toks) - 7, 7]):
            rp = TraceReplayer(str(m["folder"]), "float32", 512, page_size=m["page"], max_requests=2)
            rp.runner.cache.admit(rid)
            got, at = [], 0
            for n in cut:
                rp.runner.cache.ensure_capacity(rid, at + n)
                part = []
                rp.runner.step([StepEntry(rid, toks[at:at + n], at, list(range(n)))], layer_outputs=part)
                got.append(part)
                at += n
            assert len(got[0]) == len(want)
            for i, b in enumerate(want):
                a = torch.cat([part[i].cpu() for part in got])
                assert rel_err(a, b) < 1e-4, (which, i, cut)


def test_every_constant_and_vector_shows_in_the_logits(models):
    """The comparisons above would not notice a lost constant if it carried no weight: on the plain implementation,
    changing each moves the logits by many times the tolerance of the float32 comparisons."""
    m = models[("a", "dyn")]
    rid, toks = max(m["reqs"].items(), key=lambda kv: len(kv[1]))
    ref = m["want"][rid]
    tol = 3 * float(m["noise"][rid].max())

    def moved(config, weights=None):
        return float(sm.row_error(plain.forward(config, weights or m["weights"], toks).numpy() - ref).max())

    step = {"left.scale": lambda s: s * 1.1, "left.mask.size": lambda s: s + 1, "right.gate_cap": lambda c: c * 0.8,
            "left_scale": lambda s: s * 1.05, "right_scale": lambda s: s * 1.05, "router.top": lambda t: max(1, t - 1)}
    for path, f in step.items():
        assert moved(sm.changed(m["config"], path, f)) > 30 * tol, path
    assert moved(dict(m["config"], norm=dict(eps=1e-2))) > 30 * tol
    assert moved(dict(m["config"], logit_scale=m["config"]["logit_scale"] * 1.01)) > 30 * tol
    for name in ("l0.mix.y.b", "l0.mix.x.b", "l0.mix.conv.b", "l0.mix.ra.b", "l0.mix.ri.b", "l1.mix.right.i.b", "l1.mix.right.f.b",
                 "l0.norm1", "final.norm", "l3.mix.right.i", "l3.mix.right.f", "l0.mix.ra", "l0.mix.ri"):
        w = dict(m["weights"])
        w[name] = w[name] * 0
        assert moved(m["config"], w) > 30 * tol, name
    for name, f in (("l0.mix.lam", lambda t: t + 0.1), ("l1.mix.right.norm", lambda t: t * 0 + 1), ("l0.mix.conv", lambda t: t.roll(1, 1)),
                    ("l1.mix.right.g", lambda t: t * 0), ("l0.mlp.shared.down", lambda t: t * 0)):
        w = dict(m["weights"])
        w[name] = f(w[name])
        assert moved(m["config"], w) > 30 * tol, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, dtype):
    """A short prompt, then 150 tokens one by one: decoded keys fill page after page and chunk after chunk, states are
    carried all the way."""
    from tokasaurus_b200.engine.trace import TraceReplayer

    for which in sm.MODELS:
        m = models[(which, sm.variant(dtype))]
        toks = cuttings.random_tokens(160, m["config"]["vocab"], 7)
        mg, want = sm.margins(m["config"], m["weights"], toks)
        assert mg > (sm.MIN_MARGIN if dtype == "float32" else sm.TIER_MARGIN), which
        want = want.numpy()
        steps = cuttings.prefix_then_single({"long": toks}, tail=150)
        rp = TraceReplayer(str(m["folder"]), dtype, cuttings.max_live_tokens(steps, m["page"]), page_size=m["page"], max_requests=4)
        got = cuttings.collect(steps, [rp.run_step(st) for st in steps])
        noise = sm.rounding_noise(m["config"], m["weights"], toks, want, dtype)
        sm.check_logits(got, dict(want={"long": want}, noise={"long": noise}), dtype, "long decoding")


def plain_greedy(m, prompt, n):
    ids, out = list(prompt), []
    for _ in range(n):
        out.append(int(plain.forward(m["config"], m["weights"], ids)[-1].argmax()))
        ids.append(out[-1])
    return out


@pytest.mark.parametrize("which", ["a", "c", "d", "e"])
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_entry_point(models, graphs, which):
    """Greedy generation in float32 through ``Engine.generate``: the scheduler admits, cuts prompts into portions,
    decodes (from CUDA graphs or kernel by kernel) and frees; five requests in three slots, so slots and pages are
    handed on; prompts longer than the chunks, so pages come back while a request runs."""
    from tokasaurus_b200.engine.engine import Engine

    m = models[(which, "tier")]
    V = m["config"]["vocab"]
    prompts = [cuttings.random_tokens(n, V, 300 + n) for n in (30, 3, 61, 17, 9)]
    n_new = 10
    want = [plain_greedy(m, p, n_new) for p in prompts]
    eng = Engine(model=str(m["folder"]), dtype="float32", page_size=m["page"], kv_cache_num_tokens=512,
                 max_tokens_per_forward=24, max_seqs_per_forward=3, allocator_sanity_checks=True, use_cudagraphs=graphs)
    outs = eng.generate(prompts, max_num_tokens=n_new, ignore_eos=True)
    assert [o.completion_ids for o in outs] == want
    cache = eng.runner.cache
    assert not cache.requests and cache.num_free_pages() == [g.allocator.num_pages for g in cache.groups]


@pytest.mark.parametrize("which", ["a", "b"])
def test_bfloat16_generation_from_graphs_equals_kernel_by_kernel(models, which):
    """The serving precision: decode steps replayed from CUDA graphs choose the tokens that the same steps choose kernel by
    kernel (the same kernels on the same data), and every chosen token is near the plain statement's best at its place."""
    from tokasaurus_b200.engine.engine import Engine

    m = models[(which, "tier")]
    V = m["config"]["vocab"]
    prompts = [cuttings.random_tokens(n, V, 500 + n) for n in (70, 5, 33, 120)]
    got = []
    for graphs in (False, True):
        eng = Engine(model=str(m["folder"]), dtype="bfloat16", page_size=m["page"], kv_cache_num_tokens=1024,
                     max_tokens_per_forward=64, max_seqs_per_forward=4, allocator_sanity_checks=True, use_cudagraphs=graphs)
        got.append([o.completion_ids for o in eng.generate(prompts, max_num_tokens=12, ignore_eos=True)])
        del eng
    assert got[0] == got[1]
    for p, ids in zip(prompts, got[0]):
        logits = plain.forward(m["config"], m["weights"], p + ids[:-1])[len(p) - 1:]
        top = float(logits.abs().max())
        for i, t in enumerate(ids):
            assert float(logits[i, t]) >= float(logits[i].max()) - 0.05 * top, (which, i)


def test_command_line_generates(models, tmp_path):
    """``toka model=<folder>`` picks the model class from config.json and generates."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    m = models[("b", "tier")]
    prompt = cuttings.random_tokens(12, m["config"]["vocab"], 1)
    toka = Path(__file__).resolve().parent.parent / "bin" / "toka"
    r = subprocess.run([sys.executable, str(toka), f"model={m['folder']}", "dtype=float32", "page_size=16",
                        "kv_cache_num_tokens=256", "max_num_tokens=6", "ignore_eos=T", f"prompt_ids={json.dumps(prompt)}"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    want = plain_greedy(m, prompt, 6)
    assert json.loads(r.stdout.strip().splitlines()[-1])["completion_ids"] == want
