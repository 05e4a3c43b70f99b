"""The Safupel configuration reader and the model description built from it (no GPU): every size and constant comes
from config.json, each layer's mixer gets cache entries of its kind (two for mixers side by side), the tensor names and
shapes follow the layers, and a configuration that cannot describe a model is refused with the key that is wrong.  The
cache manager's books for a group that sees chunks.  Also the plain implementation's own mechanisms against hand-made
cases, since every GPU comparison rests on it."""

import math

import pytest
import torch

import plain_safupel as plain
from tokasaurus_b200.cache.manager import CacheManager
from tokasaurus_b200.config import lookup_architecture
from tokasaurus_b200.config.model_config import ConfigError
from tokasaurus_b200.parts.base import PagedCacheNeed, ResidualStream, StateNeed

F64 = torch.float64


def base_config():
    return dict(architecture="Safupel", vocab=97, width=48, norm=dict(eps=1e-5), logit_scale=1.7,
                layers=[dict(type="rglru", mixer=dict(width=60, blocks=3, conv=5), mlp=dict(kind="dense", ff=40)),
                        dict(type="parallel", mixer=dict(
                            left=dict(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.25, mask=dict(size=21)),
                            right=dict(heads=3, dim=10, vdim=14, gate_cap=9.0), left_scale=1.3, right_scale=0.4),
                            mlp=dict(kind="moe", expert=dict(ff=24), router=dict(experts=6, top=2), shared=dict(ff=16))),
                        dict(type="rglru", mixer=dict(width=32, blocks=1, conv=1), mlp=None)])


def test_description_follows_the_configuration():
    d = base_config()
    arch = lookup_architecture(d)
    assert arch.name == "Safupel"
    cfg = arch.parse_config(d)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.logit_scale, len(cfg.layers)) == (97, 48, 1e-5, 1.7, 3)
    model = arch.build_model(cfg)
    needs = model.cache_entries()
    assert needs[0] == StateNeed((60 * 5,)) and needs[2] == StateNeed((32,))  # S, then the convolution's last taps - 1 inputs
    assert needs[1] == PagedCacheNeed(2, 12 + 20, 21, planes=1, chunked=True)
    # the mixer beside it: S and n of three heads and their running maxima, in whole 16-byte pieces
    assert needs[3] == StateNeed((-(-(3 * 15 * 10 + 3) // 4) * 4,)) and model.stage_entries == [{}, {"right": 3}, {}]
    assert len(model.mixers()) == 4 and model.graph_safe
    names = {s.name: s for s in model.weight_specs()}
    assert names["l0.mix.y"].shape == (60, 48) and names["l0.mix.conv"].shape == (60, 5) and names["l0.mix.ra"].shape == (3, 20, 20)
    assert names["l0.mix.ri.b"].shape == (3, 20) and names["l0.mix.lam"].shape == (60,) and names["l0.mix.o"].shape == (48, 60)
    assert names["l0.mlp.up"].shape == (40, 48) and names["l0.mlp.down"].shape == (48, 40) and "l0.mlp.gate" not in names
    assert names["l1.mix.left.q"].shape == (48, 48) and names["l1.mix.left.k"].shape == (24, 48) and names["l1.mix.left.v"].shape == (40, 48)
    assert names["l1.mix.left.o"].shape == (48, 80) and names["l1.mix.right.q"].shape == (30, 48) and names["l1.mix.right.v"].shape == (42, 48)
    assert names["l1.mix.right.norm"].shape == (42,) and names["l1.mix.right.i"].shape == (3, 48) and names["l1.mix.right.f.b"].shape == (3,)
    assert names["l1.mlp.router"].role == "vector" and names["l1.mlp.shared.up"].shape == (16, 48) and "l1.mlp.e6.up" not in names
    assert "l0.norm2" not in names and names["final.norm"].shape == (48,) and names["head"].shape == (97, 48)
    left, right = model.blocks[1].mixer.left, model.blocks[1].mixer.right
    assert left.distance_bias == (2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8) and left.chunk == 21 and left.window is None
    assert right.gate_cap == 9.0 and right.q_scale == 10 ** -0.5 and right.den_eps == 1e-6
    assert (model.blocks[1].mixer.left_scale, model.blocks[1].mixer.right_scale) == (1.3, 0.4)
    ffn = model.blocks[1].ffn
    assert ffn.weigh_input and ffn.scored["renormalize"] is False and ffn.shared.inner == 16 and model.blocks[2].ffn is None
    assert model.head.norm.around_zero and model.head.norm.gain == 1.7 and model.blocks[0].norm.gain == 1.0
    mods = model.kernel_modules("float32")
    assert ("gated_recurrence.cu", None) in mods and ("attention_sink.cu", {"TKB_QK": 12, "TKB_VD": 20, "TKB_DIST": 1}) in mods


def test_defaults():
    d = base_config()
    m = d["layers"][1]["mixer"]
    for key in ("kv_heads", "vdim", "scale", "mask"):
        m["left"].pop(key)
    m["right"].pop("vdim")
    for key in ("left_scale", "right_scale"):
        m.pop(key)
    d.pop("logit_scale")
    d["layers"][1]["mlp"].pop("shared")
    cfg = lookup_architecture(d).parse_config(d)
    a, r = cfg.layers[1].mixer.left, cfg.layers[1].mixer.right
    assert (a.kv_heads, a.vdim, a.scale, a.chunk, r.vdim) == (4, 12, 1.0 / math.sqrt(12), None, 10)
    assert (cfg.layers[1].mixer.left_scale, cfg.layers[1].mixer.right_scale, cfg.logit_scale) == (1.0, 1.0, 1.0)
    model = lookup_architecture(d).build_model(cfg)
    assert model.cache_entries()[1] == PagedCacheNeed(4, 24, None, planes=1) and model.blocks[1].ffn.shared is None


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="gru"), "type"),
    (lambda d: d["layers"][0]["mixer"].update(blocks=7), "blocks"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][1]["mixer"].pop("right"), "right"),
    (lambda d: d["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][1]["mixer"]["right"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"]["right"].update(gate_cap=-1.0), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].update(left_scale="x"), "left_scale"),
    (lambda d: d["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][0]["mlp"].update(kind="glu"), "kind"),
    (lambda d: d["norm"].update(eps=0), "eps"),
    (lambda d: d.pop("width"), "width"),
])
def test_configurations_that_describe_no_model_are_refused(change, word):
    d = base_config()
    change(d)
    with pytest.raises(ConfigError) as e:
        lookup_architecture(d).parse_config(d)
    assert word in str(e.value)


def test_pages_of_earlier_chunks_come_back():
    """A group that sees chunks keeps the current chunk's pages whole, gives back those that lie before it (in one go when
    a chunk is full), and never a page that the chunk begins inside of."""
    page, chunk = 8, 20
    needs = {0: PagedCacheNeed(1, 16, chunk, planes=1, chunked=True), 1: PagedCacheNeed(1, 16, chunk, planes=1), 2: PagedCacheNeed(1, 8, None)}
    cm = CacheManager(needs, page, 40, max_requests=2, device=None)
    cm.admit("r")
    for n in (5, 19, 20, 21, 39, 40, 41, 60, 64, 79, 80, 200):
        cm.ensure_capacity("r", n)
        cm.release_behind_window("r", n)
        cm.check()
        rc = cm.requests["r"]
        for g, first in ((0, n // chunk * chunk), (1, max(0, n - chunk + 1))):
            gone = [i for i, p in enumerate(rc.tables[g]) if p < 0]
            assert gone == list(range(min(first // page, len(rc.tables[g])))), (n, g, gone)
        assert all(p >= 0 for p in rc.tables[2])
    assert needs[0].first_visible(19) == 0 and needs[0].first_visible(20) == 20 and needs[1].first_visible(20) == 1
    cm.free("r")
    assert cm.num_free_pages() == [40, 40, 40]


def test_a_stream_with_a_pair_of_updates_settles_to_their_sum():
    x = torch.randn(3, 4)
    a, b = torch.randn(2, 3, 4), torch.randn(3, 4)
    s = ResidualStream(x.clone(), (a, b))
    assert torch.allclose(s.settled(), x + a.sum(0) + b) and torch.equal(s.x, x)
    assert torch.equal(ResidualStream(x).settled(), x) and torch.allclose(ResidualStream(x, b).settled(), x + b)


def test_plain_mechanisms_on_hand_made_cases():
    t = lambda *v: torch.tensor(v, dtype=F64)  # noqa: E731
    # chunks count from position 0: positions 3 and 5 are of one chunk of 3, 2 and 3 are not
    vis = plain.visible(7, 3)
    assert vis[5].tolist() == [False, False, False, True, True, True, False] and vis[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert plain.visible(4, None).tolist() == torch.tril(torch.ones(4, 4)).bool().tolist()
    assert torch.allclose(plain.slopes(4), t(2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8))
    # with equal scores the weights fall off with the distance alone
    one = torch.zeros(3, 1, 1, dtype=F64)
    v = t(0.0, 0.0, 1.0).view(3, 1, 1)
    o = plain.distance_attention(one, one, v, 1.0, plain.visible(3, None))[2, 0, 0]
    assert abs(float(o) - 1.0 / (1 + math.exp(-2.0 ** -8) + math.exp(-2 * 2.0 ** -8))) < 1e-12
    # the last tap meets the current token, zeros before the start
    u = plain.causal_conv(t(1.0, 2.0, 4.0).view(3, 1), t(0.1, 0.5, 3.0).view(1, 3), t(7.0))
    assert torch.allclose(u[:, 0], t(10.0, 7 + 6 + 0.5, 7 + 12 + 1.0 + 0.1))
    # block-diagonal: the second part's result comes from the second part alone
    m = torch.tensor([[[1.0, 2.0], [3.0, 4.0]], [[5.0, 6.0], [7.0, 8.0]]], dtype=F64)
    y = plain.block_product(t(1.0, 10.0, 100.0, 1000.0).view(1, 4), m, torch.zeros(2, 2, dtype=F64))
    assert y[0].tolist() == [21.0, 43.0, 6500.0, 8700.0]
    assert torch.allclose(plain.diagonal_scan(t(0.5, 0.5, 0.25).view(3, 1), t(1.0, 2.0, 3.0).view(3, 1))[:, 0], t(1.0, 2.5, 3.625))
    # matrix memory, one channel: one token with gate i = 2 from m = 0: m = 2, S = k v, n = k
    q, k, v = t(2.0).view(1, 1, 1), t(3.0).view(1, 1, 1), t(5.0).view(1, 1, 1)
    o = plain.matrix_memory(q, k, v, t(2.0).view(1, 1), t(-1.0).view(1, 1))
    assert abs(float(o) - 3 * 5 * 2 / (max(6.0, math.exp(-2.0)) + 1e-6)) < 1e-12
    # a weak input: the maximum only fades by the forget gate, and the floor exp(-m) decides
    o = plain.matrix_memory(q, k, v, t(-9.0).view(1, 1), t(-1.0).view(1, 1))
    c = math.exp(-8.0)
    assert abs(float(o) - c * 30 / (max(c * 6, math.exp(1.0)) + 1e-6)) < 1e-12
    assert abs(float(plain.soft_cap(t(100.0), 4.0)) - 4.0) < 1e-12 and abs(float(plain.gelu_erf(t(1.0))) - 0.8413447460685429) < 1e-12
    # a score multiplies what goes into an expert, and is not renormalised
    w = {"router": t(0.0, 1.0).view(2, 1), "e0.gate": t(1.0).view(1, 1), "e0.up": t(1.0).view(1, 1), "e0.down": t(1.0).view(1, 1)}
    w.update({k.replace("e0", "e1"): x * 2 for k, x in w.items() if k.startswith("e0")})
    out = plain.moe_ff(t(3.0).view(1, 1), w, "", dict(router=dict(experts=2, top=1)))
    z = 3.0 / (1 + math.exp(-3.0)) * 2
    assert abs(float(out) - 2 * z / (1 + math.exp(-z)) * z) < 1e-12
    assert torch.allclose(plain.rms_norm(t(3.0, 4.0), t(0.0, 1.0), 0.0), t(3.0, 8.0) / math.sqrt(12.5))
