"""The Deletar configuration reader and the model description built from it (no GPU): every size and constant comes
from config.json, layers that read another layer's rows share its cache entry, the tensor names and shapes follow the
layers, and a configuration that cannot describe a model is refused with the key that is wrong.  The scaled rotation
frequencies.  Also the plain implementation's own mechanisms against hand-made cases, since every GPU comparison rests on it."""

import math

import pytest
import torch

import plain_deletar as plain
from tokasaurus_b200.config import lookup_architecture
from tokasaurus_b200.config.model_config import ConfigError
from tokasaurus_b200.parts import RMSNorm, RotaryEncoding, RoutedExperts, SandwichNormBlock, SinkAttention
from tokasaurus_b200.parts.base import PagedCacheNeed, ResidualStream, StateNeed, WeightSpec
from tokasaurus_b200.weights.random_init import random_tensors

F64 = torch.float64


def base_config():
    rot = dict(base=300.0, dims=6, scaling=dict(factor=3.0, low=1.0, high=2.0, original=50))
    return dict(
        architecture="Deletar", vocab=97, width=48, norm=dict(eps=1e-5), embedding=dict(scale=1.7), logit_softcap=11.0,
        layers=[dict(type="attention", mixer=dict(heads=4, kv_heads=2, dim=10, vdim=14, scale=0.4, conv=3, mask=dict(size=9),
                                                  rot=dict(base=100.0, dims=4)), mlp=dict(kind="dense", ff=40)),
                dict(type="attention_2", mixer=dict(heads=6, kv_heads=3, dim=8, vdim=8, scale=0.3, softcap=5.0,
                                                    mask=dict(size=21), rot=dict(base=200.0, dims=8)), mlp=None),
                dict(type="attention_3", mixer=dict(heads=5, kv_heads=1, dim=12, vdim=20, scale=0.2, softcap=7.0,
                                                    mask=dict(size=13), rot=dict(rot)),
                     mlp=dict(kind="moe", expert=dict(ff=24), router=dict(experts=6, top=2), shared=dict(ff=16))),
                dict(type="attention_3", mixer=dict(heads=3, kv_heads=1, dim=12, vdim=20, scale=0.5, softcap=9.0, kv_from=2,
                                                    mask=dict(size=30), rot=dict(rot)),
                     mlp=dict(kind="moe", expert=dict(ff=12), router=dict(experts=3, top=1)))])


def build(d):
    arch = lookup_architecture(d)
    return arch.build_model(arch.parse_config(d))


def test_description_follows_the_configuration():
    d = base_config()
    arch = lookup_architecture(d)
    assert arch.name == "Deletar"
    cfg = arch.parse_config(d)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.logit_softcap, len(cfg.layers)) == (97, 48, 1e-5, 1.7, 11.0, 4)
    model = arch.build_model(cfg)
    needs = model.cache_entries()
    assert needs[0] == PagedCacheNeed(2, 24, 9, planes=1) and needs[1] == PagedCacheNeed(3, 16, 21, planes=1)
    assert needs[2] == PagedCacheNeed(1, 32, 30, planes=1)  # kept as long as its wider reader needs
    assert [(c.block, c.cache, c.write_cache) for c in model.run_order] == [(0, 0, True), (1, 1, True), (2, 2, True), (3, 2, False)]
    # the convolution's last two projected rows of q, k and v
    conv = model.stage_entries[0]["conv"]
    assert needs[conv] == StateNeed((2 * (40 + 20 + 28),)) and model.stage_entries[1:] == [{}, {}, {}] and len(needs) == 4
    assert model.graph_safe
    names = {s.name: s for s in model.weight_specs()}
    assert names["l0.mix.q"].shape == (40, 48) and names["l0.mix.k"].shape == (20, 48) and names["l0.mix.v"].shape == (28, 48)
    assert names["l0.mix.q.conv"].shape == (40, 3) and names["l0.mix.v.conv"].shape == (28, 3) and names["l0.mix.o"].shape == (48, 56)
    assert "l0.mix.g" not in names and "l0.mix.q.norm" not in names and names["l0.mlp.up"].shape == (40, 48) and "l0.mlp.gate" not in names
    assert "l1.mix.v" not in names and names["l1.mix.q.b"].shape == (48,) and names["l1.mix.k.b"].shape == (24,)
    assert names["l1.mix.q.norm"].shape == (48,) and names["l1.mix.k.norm"].shape == (24,) and names["l1.mix.g"].shape == (6, 48)
    assert "l1.norm2" not in names and "l1.norm1b" in names and "l2.norm2b" in names
    assert names["l2.mix.q.norm"].shape == (12,) and names["l2.mix.k.norm"].shape == (12,)
    assert names["l2.mlp.table"] == WeightSpec("l2.mlp.table", (97, 2), role="table", below=6) and "l2.mlp.router" not in names
    assert names["l2.mlp.shared.up"].shape == (16, 48) and names["l2.mlp.e5.down"].shape == (48, 24) and "l2.mlp.e6.up" not in names
    assert not any(n in names for n in ("l3.mix.k", "l3.mix.v", "l3.mix.k.norm", "l3.mlp.shared.up")) and "l3.mix.q.norm" in names
    a, b, c, r = (blk.mixer for blk in model.blocks)
    assert (a.taps, a.window, a.softcap, a.gated, a.null_sink, a.unit_norm, a.rotary_pairs) == (3, 9, None, False, False, False, False)
    assert (b.values_are_keys, b.whole_norm, b.softcap, b.gated, b.null_sink, b.window) == (True, True, 5.0, True, False, 21)
    assert (c.whole_norm, c.null_sink, c.gated, c.own_kv, c.window, c.scale) == (False, True, True, True, 13, 0.2)
    assert (r.own_kv, r.window, r.cache_window, r.scale, r.softcap, r.n_heads) == (False, 30, 30, 0.5, 9.0, 3)
    assert c.rotary.scaling_type == "llama3" and a.rotary.scaling_type == "default"
    assert model.head.softcap == 11.0 and model.head.norm.around_zero and model.embedding.scale == 1.7
    blk = model.blocks[2]
    assert blk.ffn.by_token and blk.ffn.act == "relu2" and blk.ffn.shared.activation == "relu2" and blk.ffn.out_dtype == torch.float32
    assert blk.mixer_norm.around_zero and blk.mixer_out_norm.around_zero and blk.ffn_out_norm.around_zero and model.blocks[1].ffn is None
    mods = model.kernel_modules("float32")
    assert ("attention_sink.cu", {"TKB_QK": 10, "TKB_VD": 14, "TKB_TAPS": 3}) in mods and ("post_norm.cu", None) in mods
    assert ("attention_sink.cu", {"TKB_QK": 8, "TKB_VD": 8}) in mods and ("moe.cu", None) in mods


def test_defaults():
    d = base_config()
    m = d["layers"][2]["mixer"]
    for key in ("kv_heads", "vdim", "scale", "mask", "rot", "softcap"):
        m.pop(key)
    d["layers"] = d["layers"][:3]
    d.pop("logit_softcap"), d.pop("embedding")
    d["layers"][2]["mlp"].pop("shared")
    cfg = lookup_architecture(d).parse_config(d)
    m = cfg.layers[2].mixer
    assert (m.kv_heads, m.vdim, m.scale, m.window, m.rot, m.softcap, m.kv_from) == (5, 12, 1.0 / math.sqrt(12), None, None, None, None)
    assert (cfg.embedding_scale, cfg.logit_softcap) == (1.0, None)
    model = lookup_architecture(d).build_model(cfg)
    assert model.cache_entries()[2] == PagedCacheNeed(5, 24, None, planes=1) and model.blocks[2].ffn.shared is None
    assert model.head.softcap is None


def test_a_source_keeps_all_its_rows_for_a_reader_without_a_window():
    d = base_config()
    d["layers"][3]["mixer"].pop("mask")
    model = build(d)
    assert model.cache_entries()[2] == PagedCacheNeed(1, 32, None, planes=1) and model.blocks[2].mixer.window == 13


@pytest.mark.parametrize("change,word", [
    (lambda d: d["layers"][0].update(type="gru"), "type"),
    (lambda d: d["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda d: d["layers"][1]["mixer"].update(vdim=4), "values"),
    (lambda d: d["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda d: d["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda d: d["layers"][2]["mixer"]["rot"]["scaling"].pop("low"), "low"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda d: d["layers"][3]["mixer"].update(kv_from=1), "kv_heads"),
    (lambda d: d["layers"][3]["mixer"]["rot"].update(base=301.0), "rotation"),
    (lambda d: d["layers"].append(dict(d["layers"][3], mixer=dict(d["layers"][3]["mixer"], kv_from=3))), "kv_from"),
    (lambda d: d["layers"][2]["mlp"]["router"].update(top=7), "top"),
    (lambda d: d["layers"][0]["mlp"].update(kind="glu"), "kind"),
    (lambda d: d.update(logit_softcap=0.0), "logit_softcap"),
    (lambda d: d["norm"].update(eps=0), "eps"),
    (lambda d: d.pop("width"), "width"),
])
def test_configurations_that_describe_no_model_are_refused(change, word):
    d = base_config()
    change(d)
    with pytest.raises(ConfigError) as e:
        lookup_architecture(d).parse_config(d)
    assert word in str(e.value)


def test_parts_refuse_what_is_not_built():
    ok = dict(width=16, n_heads=2, n_kv_heads=1, dim=8, vdim=8, scale=1.0, softcap=None, window=4, norm_eps=1e-6, q_name="q",
              k_name="k", v_name="v", o_name="o", sink_name=None, unit_norm=False)
    SinkAttention(**ok)
    taps = (2, ("qc", "kc", "vc"))
    for extra in (dict(conv=(0, ("a", "b", "c"))), dict(conv=taps, bias_names=("a", "b", "c")), dict(conv=taps, values_are_keys=True),
                  dict(null_sink=True, sink_name="s"), dict(norm_over="projection"), dict(norm_over="row"), dict(cache_window=3),
                  dict(null_sink=True, weights="sigmoid")):
        with pytest.raises(ValueError):
            SinkAttention(**{**ok, **extra})
    names = lambda e: (f"e{e}.up", f"e{e}.down")  # noqa: E731
    for extra in (dict(router_name=None), dict(router_name="r", table_name="t", vocab=4), dict(router_name=None, table_name="t")):
        with pytest.raises(ValueError):
            RoutedExperts(width=16, inner=8, n_experts=3, top=1, router_bias_name=None, expert_names=names, expert="relu2", **extra)
    norm = RMSNorm(16, 1e-6, "n")
    with pytest.raises(ValueError):
        SandwichNormBlock(norm, None, norm, norm, None, None)


def test_random_tables_name_experts_that_differ_within_a_row():
    t = random_tensors([WeightSpec("t", (200, 3), role="table", below=5)], seed=1)["t"]
    assert t.dtype == torch.int32 and int(t.min()) == 0 and int(t.max()) == 4
    assert all(len(set(r)) == 3 for r in t.tolist())


def test_frequencies_scaled_by_wavelength():
    """Pairs below, between and above the two lengths, against the plain statement; also at the lengths themselves."""
    for dims, base, sc in ((20, 800.0, dict(factor=6.0, low=1.0, high=3.0, original=90)),
                           (14, 70.0, dict(factor=5.0, low=0.5, high=2.5, original=40)),
                           (64, 500000.0, dict(factor=8.0, low=1.0, high=4.0, original=8192)),
                           (8, 50.0, dict(factor=3.0, low=2.0, high=2.0, original=30))):
        r = RotaryEncoding(dims, base, "llama3", factor=sc["factor"], low_freq_factor=sc["low"], high_freq_factor=sc["high"],
                           original_max_position_embeddings=sc["original"])
        got = r.inv_freq64()
        plain_f = RotaryEncoding(dims, base).inv_freq64()
        want = plain.frequencies(dict(dims=dims, base=base, scaling=sc))
        assert torch.allclose(got, want, rtol=1e-14, atol=0)
        ratio = got / plain_f
        assert bool((ratio <= 1 + 1e-12).all()) and bool((ratio >= 1 / sc["factor"] - 1e-12).all())
        assert (float(ratio[0]), abs(float(ratio[-1]) - 1 / sc["factor"]) < 1e-12) == (1.0, True)
        if sc["high"] > sc["low"]:
            assert bool(((ratio < 0.999) & (ratio > 1.001 / sc["factor"])).any())
        assert torch.allclose(r.inv_freq().double(), got, rtol=1e-5) or sc["high"] == sc["low"]


def test_a_stream_whose_update_is_normed_settles_to_the_normed_sum():
    x, d = torch.randn(3, 4), torch.randn(2, 3, 4)
    n = RMSNorm(4, 1e-5, "n", around_zero=True)

    class Rt:
        dtype = torch.float32
    w = torch.randn(4)
    n.bind({"n": w}, Rt)
    s = ResidualStream(x.clone(), d)
    s.delta_norm = n
    want = x.double() + plain.rms_norm(d.double().sum(0), w.double(), 1e-5)
    assert torch.allclose(s.settled().double(), want, atol=1e-6) and torch.equal(s.x, x)


def test_plain_mechanisms_on_hand_made_cases():
    t = lambda *v: torch.tensor(v, dtype=F64)  # noqa: E731
    assert torch.allclose(plain.rms_norm(t(3.0, 4.0), t(0.0, 1.0), 0.0), t(3.0, 8.0) / math.sqrt(12.5))
    # the last tap meets the current token, zeros before the start
    u = plain.causal_conv(t(1.0, 2.0, 4.0).view(3, 1), t(0.1, 0.5, 3.0).view(1, 3))
    assert torch.allclose(u[:, 0], t(3.0, 6 + 0.5, 12 + 1.0 + 0.1))
    # channel 0 turns with channel 1 of two rotated ones; the third stays
    f = plain.frequencies(dict(dims=2, base=10.0))
    assert f.tolist() == [1.0]
    x = plain.rotate_half(t(1.0, 0.0, 5.0).expand(2, 1, 3), f)
    assert torch.allclose(x[1, 0], t(math.cos(1.0), math.sin(1.0), 5.0)) and torch.allclose(x[0, 0], t(1.0, 0.0, 5.0))
    vis = plain.visible(5, 2)
    assert vis[3].tolist() == [False, False, True, True, False] and plain.visible(5, 1)[4].tolist() == [False] * 4 + [True]
    assert plain.visible(3, None).tolist() == torch.tril(torch.ones(3, 3)).bool().tolist()
    # equal scores: the plain softmax averages; a key of score 0 takes its share and brings nothing
    z = torch.zeros(2, 1, 1, dtype=F64)
    v = t(2.0, 4.0).view(2, 1, 1)
    assert float(plain.softmax_attention(z, z, v, 1.0, plain.visible(2, None))[1]) == 3.0
    assert abs(float(plain.softmax_attention(z, z, v, 1.0, plain.visible(2, None), null_key=True)[1]) - 2.0) < 1e-12
    big = torch.full((1, 1, 1), 100.0, dtype=F64)
    got = plain.softmax_attention(big, big, t(1.0).view(1, 1, 1), 1.0, plain.visible(1, None), cap=3.0, null_key=True)
    assert abs(float(got) - math.exp(3.0) / (1 + math.exp(3.0))) < 1e-12  # the cap holds the score
    # values that are the keys: as projected, the bias in them, before the norm over the whole projection
    w = {"k": t(1.0, 2.0).view(2, 1), "k.b": t(0.5, -0.5), "k.norm": t(1.0, 3.0)}
    k, v = plain.keys_values(t(2.0).view(1, 1), w, "", dict(heads=2, kv_heads=2, dim=1, vdim=1), "attention_2", 0.0)
    r = math.sqrt((2.5 ** 2 + 3.5 ** 2) / 2)
    assert torch.allclose(v[0, :, 0], t(2.5, 3.5)) and torch.allclose(k[0, :, 0], t(2.5 / r, 3 * 3.5 / r))
    # a head of its own norm instead
    w = {"k": t(1.0, 2.0).view(2, 1), "v": t(7.0, 8.0).view(2, 1), "k.norm": t(3.0)}
    k, v = plain.keys_values(t(2.0).view(1, 1), w, "", dict(heads=2, kv_heads=2, dim=1, vdim=1), "attention_3", 0.0)
    assert torch.allclose(k[0, :, 0], t(3.0, 3.0)) and torch.allclose(v[0, :, 0], t(14.0, 16.0))
    # experts by token id, each of weight 1 / top, a shared one beside them
    one = lambda x: t(x).view(1, 1)  # noqa: E731
    w = {f"e{e}.{n}": one(e + 1.0) for e in range(3) for n in ("up", "down")}
    w.update({"shared.up": one(1.0), "shared.down": one(10.0), "table": torch.tensor([[0, 2], [1, 0]])})
    mlp = dict(router=dict(experts=3, top=2), shared=dict(ff=1))
    got = plain.table_moe(t(2.0, -1.0, 2.0).view(3, 1), w, "", mlp, [1, 0, 0])
    f = lambda e, x: (e + 1.0) * max(0.0, (e + 1.0) * x) ** 2  # noqa: E731
    assert torch.allclose(got[:, 0], t((f(1, 2) + f(0, 2)) / 2 + 40, 0.0, (f(0, 2) + f(2, 2)) / 2 + 40))
