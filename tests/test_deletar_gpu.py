"""The Deletar decoder on the GPU against the plain implementation in ``plain_deletar`` (float64, whole sequences, no
cache): every mechanism's kernels alone, then small random models of several shapes (``deletar_models``) through trace
replay in four cuttings and both precisions with pools that hold exactly what a trace needs, the stream layer by
layer, long decoding, and greedy generation through the engine's entry point and scheduler."""

import numpy as np
import pytest
import torch

import cuttings
import deletar_models as dm
import plain_deletar as plain

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
    """A block table of scattered pages for one request, and how many pages the pool has."""
    n_pages = -(-n_tokens // page)
    perm = np.random.default_rng(seed).permutation(n_pages + 5)[:n_pages]
    return [int(p) for p in perm], n_pages + 5


def step_tables(pieces):
    """The request tables of a step whose request r brings pieces[r] tokens: (token_seq, seq_q_start, seq_q_len)."""
    starts = [0] + [int(x) for x in np.cumsum(pieces)][:-1]
    return i32([r for r, n in enumerate(pieces) for _ in range(n)]), i32(starts), i32(list(pieces))


def csr(tables):
    return i32([0] + [int(x) for x in np.cumsum([len(t) for t in tables])]), i32([p for t in tables for p in t])


# ------------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows,H", [(1, 64), (5, 70), (3, 2048), (40, 96), (700, 132), (9, 4096), (2, 12289), (600, 4100), (1, 16384)])
def test_output_norm_sum_and_next_norm_in_one_pass(ops, dtype, rows, H):
    g = torch.Generator().manual_seed(rows + H)
    w1, w2 = torch.randn(H, generator=g) * 0.5 + 1, torch.randn(H, generator=g) * 0.5 + 1
    for slices in (0, 1, 2, 7):
        x = torch.randn(rows, H, generator=g) * 2
        y = torch.randn((slices, rows, H) if slices else (rows, H), generator=g) * 0.02  # (eps carries weight)
        e1, e2 = 1e-4, 1e-6
        total = x.double() + plain.rms(y.double().sum(0) if slices else y.double(), e1) * w1.double()
        xd, out = x.to(DEV), torch.empty(rows, H, dtype=DT[dtype], device=DEV)
        ops.norm_add_norm(xd, y.to(DEV), w1.to(DEV), e1, w2.to(DEV), e2, out)
        assert rel_err(xd.cpu(), total) < 1e-6
        assert rel_err(out.float().cpu(), plain.rms(total, e2) * w2.double()) < (2e-6 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("n", [1, 3, 4, 77, 5000])
def test_soft_cap(ops, n):
    for cap in (0.7, 30.0):
        z = torch.randn(3, n, generator=torch.Generator().manual_seed(n)) * 2 * cap
        got = z.to(DEV)
        ops.soft_cap(got, cap)
        assert rel_err(got.cpu(), plain.soft_cap(z.double(), cap)) < 1e-6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,inner", [(1, 64, 40), (7, 96, 72), (16, 70, 26), (40, 128, 96), (200, 96, 136), (130, 70, 26)])
def test_ungated_feed_forward_with_the_squared_relu(ops, dtype, T, H, inner):
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import SquaredReluMLP

    g = torch.Generator().manual_seed(T + inner)
    w = {"up": (torch.randn(inner, H, generator=g) * 0.25).bfloat16(), "down": (torch.randn(H, inner, generator=g) * 0.2).bfloat16()}
    h = torch.randn(T, H, generator=g).to(DT[dtype])
    part = SquaredReluMLP(H, inner, "up", "down")
    part.bind({k: v.to(DEV, DT[dtype]) for k, v in w.items()}, Runtime.make(DEV, dtype))
    got = part.forward(None, h.to(DEV))
    assert got.dtype == torch.float32
    got = (got.sum(0) if got.dim() == 3 else got).cpu()
    want = plain.squared_relu_ff(h.double(), {k: v.double() for k, v in w.items()}, "")
    assert rel_err(got, want) < (1e-5 if dtype == "float32" else 1.5e-2)


class TokenStep:
    """What experts by token id look at of a step: ids, some of them the request's last sampled token, padding behind."""

    def __init__(self, V, T, seed, pad=0):
        r = np.random.default_rng(seed)
        n_req = max(1, T // 3)
        self.ids = r.integers(0, V, T)
        seq = np.sort(r.integers(0, n_req, T))
        slots = r.permutation(n_req + 2)[:n_req]
        sampled = r.random(T) < 0.3
        last = r.integers(0, V, n_req + 2)
        for t in np.nonzero(sampled)[0]:
            self.ids[t] = last[slots[seq[t]]]
        given = np.where(sampled, -1, self.ids)
        self.n_tokens = T + pad
        self.token_ids = i32(np.concatenate([given, np.full(pad, V + 7)]))
        self.token_seq = i32(np.concatenate([seq, np.full(pad, -1)]))
        self.seq_slot, self.last_token = i32(slots), i32(last)
        self.status = torch.zeros(1, dtype=torch.int32, device=DEV)


def test_a_table_gives_each_token_its_experts(ops):
    V, E, top, T = 50, 7, 3, 90
    table = torch.rand(V, E, generator=torch.Generator().manual_seed(1)).argsort(-1)[:, :top].to(torch.int32)
    st = TokenStep(V, T, 3, pad=6)
    for rows in (None, [5, 0, 89, 44], [T + 1, 3]):
        n = st.n_tokens if rows is None else len(rows)
        idx, w = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
        ops.moe_table(table.to(DEV), E, st.token_ids, st.token_seq, st.seq_slot, st.last_token,
                      None if rows is None else i32(rows), idx, w, st.status)
        for r, t in enumerate(range(st.n_tokens) if rows is None else rows):
            if t < T:
                assert idx[r].tolist() == table[st.ids[t]].tolist() and torch.allclose(w[r].cpu(), torch.full((top,), 1 / 3))
            else:
                assert idx[r].tolist() == [-1] * top and w[r].tolist() == [0.0] * top
    assert int(st.status.item()) == 0  # (a padding token's id is nobody's business)
    st.token_ids[4] = V
    ops.moe_table(table.to(DEV), E, st.token_ids, st.token_seq, st.seq_slot, st.last_token, i32([4, 5]), idx[:2], w[:2], st.status)
    assert int(st.status.item()) == 1 and idx[0].tolist() == [-1] * top and idx[1].tolist() == table[st.ids[5]].tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,E,top,H,inner,shared", [(3, 4, 2, 64, 40, 24), (5, 6, 1, 96, 32, None), (70, 8, 4, 128, 64, 64),
                                                    (400, 5, 5, 96, 72, 40), (150, 3, 2, 128, 64, None), (33, 2, 1, 70, 22, 26),
                                                    (700, 4, 1, 70, 22, None)])
def test_experts_chosen_by_token_id(ops, dtype, T, E, top, H, inner, shared):
    """The part: few rows, tiled, and in bfloat16 the grouped tensor-core products, beside a shared expert; all of a step's
    rows, and a cut-down set of them."""
    from tokasaurus_b200.engine.runtime import Runtime
    from tokasaurus_b200.parts import RoutedExperts, SquaredReluMLP

    V = 61
    g = torch.Generator().manual_seed(T + E)
    w = {"table": torch.rand(V, E, generator=g).argsort(-1)[:, :top].to(torch.int32)}
    for e in list(range(E)) + (["s"] if shared else []):
        p, n = (f"e{e}", inner) if e != "s" else ("shared", shared)
        w[p + ".up"], w[p + ".down"] = torch.randn(n, H, generator=g) * 0.25, torch.randn(H, n, generator=g) * 0.25
    w = {k: v if k == "table" else v.to(torch.bfloat16).float() for k, v in w.items()}
    mlp = dict(router=dict(experts=E, top=top), shared=dict(ff=shared) if shared else None)
    h = torch.randn(T, H, generator=g).to(DT[dtype])
    sh = SquaredReluMLP(H, shared, "shared.up", "shared.down") if shared else None
    part = RoutedExperts(H, inner, E, top, None, None, lambda e: (f"e{e}.up", f"e{e}.down"), sh, expert="relu2",
                         out_dtype=torch.float32, table_name="table", vocab=V)
    part.bind({k: v.to(DEV) if k == "table" else v.to(DEV, DT[dtype]) for k, v in w.items()}, Runtime.make(DEV, dtype))
    st = TokenStep(V, T, T)
    got = part.forward(st, h.to(DEV))
    w64 = {k: v if k == "table" else v.double() for k, v in w.items()}
    want = plain.table_moe(h.double(), w64, "", mlp, st.ids)
    tol = 3e-5 if dtype == "float32" else 2e-2
    assert got.dtype == torch.float32 and rel_err(got.cpu(), want) < tol
    rows = sorted({0, T - 1, T // 2, T // 3})
    cut = part.forward(st, h[rows].to(DEV).contiguous(), rows=i32(rows)).cpu()
    assert rel_err(cut, want[rows]) < tol
    if len(rows) != T:
        with pytest.raises(ValueError):
            part.forward(st, h[rows].to(DEV).contiguous())


def make_rotary(dims, base):
    from tokasaurus_b200.parts import RotaryEncoding
    return RotaryEncoding(dims, base).inv_freq64().to(DEV)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,e,taps,rot,norm,own", [
    (4, 2, 16, 32, 4, 8, False, True), (3, 1, 24, 40, 3, 24, True, True), (2, 2, 10, 13, 6, 6, False, True),
    (8, 2, 128, 128, 3, 64, False, True), (5, 1, 64, 16, 2, 0, True, True), (6, 3, 32, 32, 5, 32, False, False),
    (1, 1, 300, 20, 3, 100, True, True), (2, 1, 16, 64, 1, 16, False, True)])
def test_convolution_behind_the_projections(ops, dtype, H, G, d, e, taps, rot, norm, own):
    """q, k and v through a causal convolution, then (optionally) the norm and the rotation: requests side by side, portions
    down to one and two tokens that end within and across the kernel's token groups, steps of single tokens, padding
    tokens, a slot taken over.  The state is the last projected rows, bit for bit, and how a request was cut does not
    change a bit of what comes out."""
    page, eps = 8, 1e-5
    C = H * d + (G * (d + e) if own else 0)
    g = torch.Generator().manual_seed(C + taps)
    w = torch.randn(C, taps, generator=g) * 0.6
    nw = torch.rand(2, d, generator=g) + 0.5
    freq = make_rotary(rot, 300.0) if rot else None
    reqs = {r: torch.randn(n, C + 3, generator=torch.Generator().manual_seed(i)) for i, (r, n) in enumerate(dict(a=500, b=90, c=9, d=61, e=1).items())}
    plan = [{"a": 300, "b": 3}, {"a": 2, "b": 1, "c": 1, "e": 1}, {"c": 5, "b": 70, "a": 1}, {"a": 1, "b": 1, "c": 1}, {"b": 15, "c": 2},
            {"a": 130, "d": 40}, {"d": 2, "a": 2}, {"d": 1, "a": 1}, {"a": 63, "d": 18}]
    slots = {"a": 2, "b": 0, "c": 1, "d": 0, "e": 3}  # d takes over b's slot

    def turned(x, T, heads):
        x = x.view(T, heads, d)
        return plain.rotate_half(x, freq.cpu()) if rot else x

    def want(p):
        T = p.shape[0]
        u = plain.causal_conv(p[:, :C].double(), w.double())
        q = u[:, :H * d].view(T, H, d)
        q = turned(plain.rms(q, eps) * nw[0].double() if norm else q, T, H)
        if not own:
            return q, None, None
        k = u[:, H * d:(H + G) * d].view(T, G, d)
        return q, turned(plain.rms(k, eps) * nw[1].double() if norm else k, T, G), u[:, (H + G) * d:].view(T, G, e)

    tables, pool = {}, 0
    for r, p in reqs.items():
        n = -(-p.shape[0] // page)
        tables[r] = [pool + int(x) for x in np.random.default_rng(n).permutation(n)]
        pool += n
    state = torch.full((5, max(1, (taps - 1) * C)), float("nan"), device=DEV)
    cache = torch.full((pool + 1, G, page, d + e), float("nan"), dtype=DT[dtype], device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    at, outs = dict.fromkeys(reqs, 0), {r: [] for r in reqs}

    def run(step, state, cache, pad=0):
        rows = torch.cat([reqs[r][at[r]:at[r] + n] for r, n in step.items()] + [torch.full((pad, C + 3), float("nan"))]).to(DEV)
        seq, q_start, q_len = step_tables(list(step.values()))
        pos = i32([p for r, n in step.items() for p in range(at[r], at[r] + n)] + [0] * pad)
        indptr, ids = csr([tables[r][:-(-(at[r] + n) // page)] for r, n in step.items()])
        q = torch.full((rows.shape[0], H * d), 7.0, dtype=DT[dtype], device=DEV)
        ops.sink_attn_conv_prep(rows, w.to(DEV), state if taps > 1 else None, norm, eps, q, cache, pos, torch.cat([seq, i32([-1] * pad)]),
                                i32([slots[r] for r in step]), q_start, q_len, len(step), any(n > 1 for n in step.values()),
                                indptr, ids, H, G, d, e, page, own, True, status, norm_w=nw.to(DEV) if norm else None,
                                rot_freq=freq, rot_dims=rot, own_kv=own)
        return q

    for i, step in enumerate(plan):
        for r in step:
            if at[r] == 0:
                state[slots[r]].zero_()
        q = run(step, state, cache, pad=2 if i % 2 else 0)
        assert bool((q[sum(step.values()):] == 7.0).all())
        lo = 0
        for r, n in step.items():
            outs[r].append(q[lo:lo + n].cpu())
            at[r] += n
            lo += n
            kept = torch.cat([torch.zeros(taps, C), reqs[r][:at[r], :C]])[-(taps - 1):] if taps > 1 else None
            assert taps == 1 or torch.equal(state[slots[r], :(taps - 1) * C].cpu().view(taps - 1, C), kept), (r, at[r])
    assert int(status.item()) == 0 and bool(torch.isnan(state[4]).all()) and bool(torch.isnan(cache[pool].float()).all())
    tol = 2e-5 if dtype == "float32" else 6e-3
    for r, p in reqs.items():
        n = p.shape[0]
        assert at[r] == n
        q, k, v = want(p)
        assert rel_err(torch.cat(outs[r]).float(), q.reshape(n, H * d)) < tol, r
        if own:
            kept = cache[[tables[r][t // page] for t in range(n)], :, [t % page for t in range(n)]].float().cpu()
            assert rel_err(kept[..., :d], k) < tol and rel_err(kept[..., d:], v) < tol, r
    # the same request whole: not a bit differs
    at["a"] = 0
    other = torch.zeros_like(state), torch.zeros_like(cache)
    q = run({"a": 500}, *other)
    assert torch.equal(q.cpu(), torch.cat(outs["a"]))
    mine = [t for t in tables["a"]]
    if own:
        same = torch.nan_to_num(cache[mine].float()) == torch.nan_to_num(other[1][mine].float())
        assert bool(same.flatten(2).all() if 500 % page == 0 else same[:500 // page].all())
    assert taps == 1 or torch.equal(other[0][2], state[2])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,rot,own,bias", [(6, 2, 24, 24, True, True), (2, 2, 64, 32, True, False), (3, 3, 9, 2, True, True),
                                                (16, 4, 128, 128, True, True), (5, 1, 32, 0, False, True)])
def test_norm_over_the_whole_projection(ops, dtype, H, G, d, rot, own, bias):
    """One root mean square for all of q and one for all of k (heads of very different sizes), biases under it, the keys as
    projected for values, a layer that projects q alone."""
    page, eps, T = 8, 1e-5, 37
    C = (H + G) * d if own else H * d
    g = torch.Generator().manual_seed(C)
    raw = torch.randn(T, C + 5, generator=g)
    raw[:, :C] *= torch.repeat_interleave(torch.logspace(-1, 1, C // d), d)
    b = torch.randn(C, generator=g) if bias else None
    w = torch.rand(C, generator=g) + 0.5
    x = raw[:, :C].double() + (b.double() if bias else 0.0)
    freq = make_rotary(rot, 90.0) if rot else None
    turn = lambda t: plain.rotate_half(t, freq.cpu()) if rot else t  # noqa: E731
    q = turn((plain.rms(x[:, :H * d], eps) * w[:H * d].double()).view(T, H, d))
    table, n_pages = paged(T, page, 3)
    cache = torch.full((n_pages, G, page, 2 * d), float("nan"), dtype=DT[dtype], device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.empty(T, H * d, dtype=DT[dtype], device=DEV)
    seq, _, _ = step_tables([T])
    indptr, ids = csr([table])
    ops.sink_attn_prep(raw.to(DEV), b.to(DEV) if bias else None, True, eps, out, cache, i32(range(T)), seq, indptr, ids, H, G, d, d,
                       page, own, status, norm_w=w.to(DEV), rot_freq=freq, rot_dims=rot, values_are_keys=own, whole_norm=True, own_kv=own)
    tol = 1e-5 if dtype == "float32" else 6e-3
    assert int(status.item()) == 0 and rel_err(out.float().cpu(), q.reshape(T, H * d)) < tol
    if not own:
        assert bool(torch.isnan(cache.float()).all())
        return
    k = turn((plain.rms(x[:, H * d:], eps) * w[H * d:].double()).view(T, G, d))
    kept = cache[[table[t // page] for t in range(T)], :, [t % page for t in range(T)]].float().cpu()
    assert rel_err(kept[..., :d], k) < tol and rel_err(kept[..., d:], x[:, H * d:].view(T, G, d)) < tol


def window_case(raw, H, G, d, e, scale, window, cap, null, gate):
    """Attention from raw projections [n, q | k | v] with plain's building blocks; gate logits [n, H] or None."""
    n = raw.shape[0]
    q = raw[:, :H * d].double().view(n, H, d)
    k = raw[:, H * d:(H + G) * d].double().view(n, G, d).repeat_interleave(H // G, dim=1)
    v = raw[:, (H + G) * d:(H + G) * d + G * e].double().view(n, G, e).repeat_interleave(H // G, dim=1)
    o = plain.softmax_attention(q, k, v, scale, plain.visible(n, window), cap, null)
    if gate is not None:
        o = o * torch.sigmoid(gate.double())[:, :, None]
    return o.reshape(n, H * e)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,e,page,H,G,window,cap,null", [
    (16, 32, 16, 4, 2, 37, 20.0, True), (32, 64, 16, 20, 1, 64, 12.0, True), (24, 40, 8, 2, 2, 50, None, False),
    (64, 64, 16, 2, 2, 16, 9.0, True), (48, 80, 16, 6, 3, 130, 30.0, False), (10, 13, 8, 3, 3, 40, 15.0, True),
    (128, 128, 16, 4, 1, 100, 20.0, True), (96, 96, 16, 4, 2, 65, 20.0, True), (32, 32, 16, 2, 1, 1, 5.0, True),
    (32, 32, 8, 2, 1, None, 20.0, False)])
def test_windows_capped_scores_the_null_sink_and_the_output_gate(ops, dtype, d, e, page, H, G, window, cap, null):
    """Made-up keys that made-up queries score far above all others stand at the window's first position (just inside) and
    one before it (just outside), asked for in a portion and by single tokens, without a window far away.  In one piece, in
    portions that end at and within pages, and token by token, beside a second request of one token; on the FP32 pipes and
    (in bfloat16, for sizes they take) on the tensor cores.  A second reader with a narrower window of its own reads the
    same rows."""
    n = 300
    g = torch.Generator().manual_seed(d + page + H)
    C = (H + G) * d + G * e
    scale = d ** -0.5
    raw = torch.randn(n, C, generator=g)
    gate = torch.randn(n, H, generator=g) * 2
    u = torch.randn(d, generator=g).sign() * (14.0 / d ** 0.5) ** 0.5  # aligned pairs score 14
    wd = window or 230
    pairs = [(q - wd + 1, q) for q in (wd + 7, n - 4)] + [(q - wd, q) for q in (wd + 20, n - 2)]  # inside, then outside
    for key, query in pairs:
        raw[key, H * d:(H + G) * d] = u.repeat(G)
        raw[query, :H * d] = u.repeat(H)
    if wd < 10:
        raw[:, :(H + G) * d] = torch.randn(n, (H + G) * d, generator=g)
    raw = raw.to(torch.bfloat16).float() if dtype == "bfloat16" else raw
    want = window_case(raw, H, G, d, e, scale, window, cap, null, gate)
    if window is not None and window > 10:  # the plain result at these queries rests on the window's edges
        for other, rows in ((window - 1, (pairs[0][1], pairs[1][1])), (window + 1, (pairs[2][1], pairs[3][1]))):
            moved = window_case(raw, H, G, d, e, scale, other, cap, null, gate)
            assert all(float((moved[r] - want[r]).abs().max()) > 0.1 * float(want[r].abs().max()) for r in rows)
    if null:  # a one in the denominator: leaving it out shows
        moved = window_case(raw, H, G, d, e, scale, window, cap, False, gate)
        assert float((moved - want).abs().max()) > (0.02 if window == 1 else 1e-3) * float(want.abs().max())
    narrow = None if window is None or window < 5 else window // 2
    want2 = window_case(raw, H, G, d, e, scale, narrow, cap, null, None) if narrow else None
    table, n_pages = paged(n, page, 7)
    beside_raw = torch.randn(1, C, generator=g).to(torch.bfloat16).float()
    sinks = torch.zeros(H, device=DEV) if null else None
    tol = 2e-5 if dtype == "float32" else 2e-2
    for cut in ([n], [page + 1, 3, 2, 2 * page, 2], [wd + 5, 1, 1, 1, 1, 2]):
        cut = cut + [min(64, n - sum(cut))] if sum(cut) < n else [n]
        if sum(cut) < n:
            cut += ([n - sum(cut) - 6] if n - sum(cut) > 6 else []) + [1] * min(6, n - sum(cut))
        assert sum(cut) == n
        for tc in ([False, True] if ops.can_use_attn_sink_tc(DT[dtype], d, e) else [False]):
            cache = torch.full((n_pages + 1, G, page, d + e), float("nan"), dtype=DT[dtype], device=DEV)
            status = torch.zeros(1, dtype=torch.int32, device=DEV)
            at, outs, outs2 = 0, [], []
            for m in cut:
                rows, gr = torch.cat([raw[at:at + m], beside_raw]), torch.cat([gate[at:at + m], gate[:1]])
                T = m + 1
                seq, q_start, q_len = step_tables([m, 1])
                pos = i32(list(range(at, at + m)) + [0])
                indptr, ids = csr([table[:-(-(at + m) // page)], [n_pages]])
                q = torch.empty(T, H * d, dtype=DT[dtype], device=DEV)
                wide = torch.cat([rows, torch.full((T, 2), float("nan")), gr, torch.zeros(T, 1)], dim=1).to(DEV)
                ops.sink_attn_prep(wide, None, False, 1e-6, q, cache, pos, seq, indptr, ids, H, G, d, e, page, True, status)
                for w, g_in, keep in ((window, wide[:, C + 2:C + 2 + H], outs), (narrow, None, outs2)):
                    if keep is outs2 and not narrow:
                        continue
                    out = torch.empty(T, H * e, dtype=DT[dtype], device=DEV)
                    if tc:
                        ops.attn_sink_tc(q, out, cache, q_start, q_len, i32([at + m, 1]), indptr, ids, 2, sinks, H, G, d, e, page,
                                         scale, cap, w, status, gate=g_in)
                    else:
                        ops.attn_sink(q, out, cache, seq, pos, indptr, ids, None, T, sinks, H, G, d, e, page, scale, cap, w, status,
                                      gate=g_in)
                    keep.append(out[:m].float().cpu())
                    if g_in is not None:
                        alone = window_case(beside_raw, H, G, d, e, scale, w, cap, null, gate[:1])
                        assert rel_err(out[m:].float().cpu(), alone) < tol
                at += m
            assert int(status.item()) == 0
            assert row_err(torch.cat(outs), want) < tol, (tc, cut)
            if narrow:
                assert row_err(torch.cat(outs2), want2) < tol, (tc, cut)
            if not tc:  # only some rows, named
                picked = [0, n - 1, wd + 7 if wd + 7 < n else 5]
                # (every row's query again, from the whole request)
                qa = torch.empty(n, H * d, dtype=DT[dtype], device=DEV)
                full = torch.cat([raw, gate], dim=1).to(DEV)
                sq, _, _ = step_tables([n])
                ip, idl = csr([table])
                ops.sink_attn_prep(full, None, False, 1e-6, qa, cache, i32(range(n)), sq, ip, idl, H, G, d, e, page, False, status)
                out = torch.empty(3, H * e, dtype=DT[dtype], device=DEV)
                ops.attn_sink(qa, out, cache, sq, i32(range(n)), ip, idl, i32(picked), 3, sinks, H, G, d, e, page, scale, cap, window,
                              status, gate=full[:, C:])
                assert row_err(out.float().cpu(), want[picked]) < tol


# ------------------------------------------------------------------------------------------------ whole models
@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return dm.make_models(tmp_path_factory.mktemp("deletar_models"))


CUTS = dict(whole=cuttings.whole, prefix_then_single=cuttings.prefix_then_single,
            changing_portions=cuttings.changing_portions, mixed=cuttings.mixed)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", list(CUTS))
@pytest.mark.parametrize("which", list(dm.MODELS))
def test_cuttings_match_plain(models, which, cut, dtype):
    """Whole prompts, prompts then single tokens, portions of changing size down to one and two tokens, and up to four
    requests side by side in four slots, in a pool that holds exactly what the trace needs: pages and slots are used again
    (pages behind the windows within a request's own life, too), and a later request must see nothing of an earlier one's
    keys and states."""
    from tokasaurus_b200.engine.trace import TraceReplayer

    m = models[which]
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
                assert all((p < 0) == (i < first) for i, p in enumerate(rc.tables[gi])), "pages behind the window go back, others stay"
    assert not cache.requests and cache.num_free_pages() == [g.allocator.num_pages for g in cache.groups]
    dm.check_logits(cuttings.collect(steps, outs), m["want"], m["noise"][dtype], dtype, cut)
    if cut == "mixed":
        assert any(len(v) > 1 for v in users.values()), "no slot was used by two requests"
        assert any(len(v) > 1 for v in owners.values()), "no page was used by two requests"


def test_layer_by_layer(models):
    """The residual stream after every layer, float32, one prompt in one step and in two."""
    from tokasaurus_b200.engine.batch import StepEntry
    from tokasaurus_b200.engine.trace import TraceReplayer

    for which, m in models.items():
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


def test_only_the_wanted_rows(models):
    """A step that wants some of its rows (the last layer then runs for these alone, and its experts must know which tokens
    they belong to) gives what a step that wants them all gives there."""
    from tokasaurus_b200.engine.trace import TraceReplayer

    for which, m in models.items():
        toks = max(m["reqs"].values(), key=len)
        n = len(toks)
        want = [0, n // 3, n - 2]
        other = m["reqs"][which + "1"]
        for dtype in ("float32", "bfloat16"):
            rp = TraceReplayer(str(m["folder"]), dtype, 1024, page_size=m["page"], max_requests=4)
            step = dict(step=0, entries=[dict(id="x", tokens=toks, want=want), dict(id="y", tokens=other, want=[len(other) - 1])], end=["x", "y"])
            got = rp.run_step(step)
            ref = plain.forward(m["config"], m["weights"], toks).numpy()[want]
            ref = np.concatenate([ref, plain.forward(m["config"], m["weights"], other).numpy()[-1:]])
            noise = max(float(v.max()) for v in m["noise"][dtype].values())
            assert float(dm.row_error(got - ref).max()) < 4 * noise, (which, dtype)


def test_every_constant_and_vector_shows_in_the_logits(models):
    """The comparisons above would not notice a lost constant if it carried no weight: on the plain implementation,
    changing each moves the logits by many times the tolerance of the float32 comparisons."""
    m = models["a"]
    rid, toks = max(m["reqs"].items(), key=lambda kv: len(kv[1]))
    ref = m["want"][rid]
    tol = 3 * float(m["noise"]["float32"][rid].max())

    def moved(config, weights=None):
        return float(dm.row_error(plain.forward(config, weights or m["weights"], toks).numpy() - ref).max())

    step = {"scale": lambda s: s * 1.05, "softcap": lambda c: c * 0.8, "mask.size": lambda s: s + 1, "rot.base": lambda b: b * 1.2,
            "rot.scaling.factor": lambda f: f * 1.3, "rot.scaling.original": lambda o: o * 2, "rot.scaling.high": lambda h: h + 1}
    for path, f in step.items():
        assert moved(dm.changed(m["config"], path, f)) > 30 * tol, path
    assert moved(dict(m["config"], norm=dict(eps=1e-2))) > 30 * tol
    assert moved(dict(m["config"], embedding=dict(scale=m["config"]["embedding"]["scale"] * 1.05))) > 30 * tol
    assert moved(dict(m["config"], logit_softcap=m["config"]["logit_softcap"] * 1.1)) > 30 * tol
    for name in ("l1.mix.q.b", "l1.mix.k.b", "l1.mix.g", "l2.mix.g", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l2.norm1b",
                 "final.norm"):
        w = dict(m["weights"])
        w[name] = w[name] * 0
        assert moved(m["config"], w) > 30 * tol, name
    for name, f in (("l0.mix.q.conv", lambda t: t.roll(1, 1)), ("l0.mix.v.conv", lambda t: t.roll(1, 1)), ("l4.mix.k.conv", lambda t: t.flip(1)),
                    ("l1.mix.q.norm", lambda t: t * 0 + 1), ("l1.mix.k.norm", lambda t: t.roll(24)), ("l3.mix.q.norm", lambda t: t.abs()),
                    ("l1.mlp.table", lambda t: (t + 1) % 6), ("l1.mlp.shared.down", lambda t: t * 0)):
        w = dict(m["weights"])
        w[name] = f(w[name])
        assert moved(m["config"], w) > 30 * tol, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(models, dtype):
    """A short prompt, then 150 tokens one by one: decoded keys fill page after page and fall out of the windows, the
    convolutions' states are carried all the way."""
    from tokasaurus_b200.engine.trace import TraceReplayer

    for which, m in models.items():
        toks = cuttings.random_tokens(160, m["config"]["vocab"], 7)
        want = plain.forward(m["config"], m["weights"], toks).numpy()
        steps = cuttings.prefix_then_single({"long": toks}, tail=150)
        rp = TraceReplayer(str(m["folder"]), dtype, cuttings.max_live_tokens(steps, m["page"]), page_size=m["page"], max_requests=4)
        got = cuttings.collect(steps, [rp.run_step(st) for st in steps])
        noise = dm.rounding_noise(m["config"], m["weights"], toks, want, dtype)
        dm.check_logits(got, {"long": want}, {"long": noise}, dtype, f"long decoding ({which})")


def plain_greedy(m, prompt, n):
    ids, out = list(prompt), []
    for _ in range(n):
        out.append(int(plain.forward(m["config"], m["weights"], ids)[-1].argmax()))
        ids.append(out[-1])
    return out


@pytest.mark.parametrize("which", list(dm.MODELS))
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_entry_point(models, graphs, which):
    """Greedy generation in float32 through ``Engine.generate``: the scheduler admits, cuts prompts into portions,
    decodes (from CUDA graphs or kernel by kernel; a decoding token's id is on the device alone, where its experts find it)
    and frees; five requests in three slots, so slots and pages are handed on; prompts longer than the windows, so pages
    come back while a request runs."""
    from tokasaurus_b200.engine.engine import Engine

    m = models[which]
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

    m = models[which]
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

    m = models["b"]
    prompt = cuttings.random_tokens(12, m["config"]["vocab"], 1)
    toka = Path(__file__).resolve().parent.parent / "bin" / "toka"
    r = subprocess.run([sys.executable, str(toka), f"model={m['folder']}", "dtype=float32", "page_size=16",
                        "kv_cache_num_tokens=256", "max_num_tokens=6", "ignore_eos=T", f"prompt_ids={json.dumps(prompt)}"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    want = plain_greedy(m, prompt, 6)
    assert json.loads(r.stdout.strip().splitlines()[-1])["completion_ids"] == want
