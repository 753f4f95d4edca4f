"""Lanirax on the CPU: the typed configuration, the model's tensors, caches and schedule, and the plain implementation's own
consistency (stretched frequencies, rotation, temperature, slopes, window, sink, recurrence, mixture), which the GPU tests lean on."""
import json
import math

import pytest
import torch

import plain_lanirax as plain
from lanirax_cases import CASES, SINGLE, attention, config, moe, pair, shared, stretched, write_model


def build(raw, max_positions=256):
    import carbon_engine_b200.models  # noqa: F401
    from carbon_engine_b200.config.registry import resolve_architecture
    arch = resolve_architecture(raw)
    cfg = arch.parse_config(dict(raw))
    return cfg, arch.build_model(cfg, max_positions)


def test_config_round_trip_registry_and_schedule():
    from carbon_engine_b200.config.lanirax import LaniraxConfig
    from carbon_engine_b200.parts.model import LayerCall
    for name, raw in {**CASES, **SINGLE}.items():
        cfg, model = build(raw)
        assert isinstance(cfg, LaniraxConfig) and cfg.architecture == "Lanirax"
        assert LaniraxConfig.from_dict(json.loads(json.dumps(cfg.to_json_dict()))) == cfg, name
        owners = [l for l in raw["layers"] if l.get("weights_of") is None]
        assert len(model.blocks) == len(owners) and len(model.schedule) == len(raw["layers"])
    _, model = build(CASES["A"])
    assert model.schedule == [LayerCall(0, 0, True), LayerCall(1, 1, True), LayerCall(0, 2, True), LayerCall(2, 3, True)]
    _, model = build(CASES["B"])            # layer 0 runs the weights of layer 2, which comes later
    assert [c.block for c in model.schedule] == [1, 0, 1, 2] and [c.cache for c in model.schedule] == [0, 1, 2, 3]


@pytest.mark.parametrize("bad, text", [
    (lambda r: r["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda r: r["layers"][1]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(kv_heads=3), "not a multiple"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(vdim=20), "projected keys"),
    (lambda r: r["layers"][0]["mixer"]["left"].update(mask={"size": 0}), "size"),
    (lambda r: r["layers"][0]["mixer"]["right"].update(conv=0), "conv"),
    (lambda r: r["layers"][1]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda r: r["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda r: r["layers"][1]["mlp"]["router"].update(top=10), "top=10 of 9"),
    (lambda r: r["layers"][1]["mlp"].update(kind="dense"), "mlp"),
    (lambda r: r.update(norm={"eps": 0.0}), "positive"),
    (lambda r: r.pop("postln_alpha"), "postln_alpha"),
    (lambda r: r["layers"][2].update(weights_of=9), "weights_of"),
    (lambda r: (r["layers"][0].update(weights_of=2)), "circle"),
])
def test_config_errors_name_the_key(bad, text):
    from carbon_engine_b200.config.base import ConfigError
    from carbon_engine_b200.config.lanirax import LaniraxConfig
    raw = json.loads(json.dumps(CASES["A"]))
    bad(raw)
    with pytest.raises(ConfigError, match=text):
        LaniraxConfig.from_dict(raw)


def test_tensors_and_caches():
    from carbon_engine_b200.parts.base import BundleCacheSpec, PagedCacheSpec, StateCacheSpec
    cfg, model = build(CASES["A"])
    names = {s.name: s.shape for s in model.all_tensor_specs()}
    assert names["embed.norm"] == (40,) and names["final.norm"] == (40,) and names["head"] == (97, 40)
    assert names["l0.mix.left.q"] == (64, 40) and names["l0.mix.left.k"] == (32, 40) and names["l0.mix.left.sink"] == (4,)
    assert "l0.mix.left.v" not in names and "l0.mix.left.q.norm" not in names
    assert names["l0.mix.right.v.conv"] == (56, 4) and names["l0.mix.right.a"] == (4, 40) and names["l0.mix.right.norm"] == (14,)
    assert names["l0.mix.left.out"] == names["l0.mix.right.out"] == names["l0.norm1"] == names["l0.norm2"] == (40,)
    assert names["l1.mix.q.norm"] == names["l1.mix.k.norm"] == (12,) and names["l1.mix.v"] == (40, 40) and names["l1.mix.o"] == (40, 80)
    assert names["l1.mlp.router"] == (9, 40) and names["l1.mlp.router.b"] == (9,) and names["l1.mlp.e8.down"] == (40, 10)
    assert not any(n.startswith("l2.") for n in names) and "l3.norm2" not in names and "l3.norm1" in names
    layout = dict(model.cache_layout())
    assert isinstance(layout[0], BundleCacheSpec) and layout[0].main == PagedCacheSpec(2, 16, 9, None, v_heads=2, v_head_dim=16)
    assert dict(layout[0].extra) == {"1.state": StateCacheSpec((4, 10, 14), torch.float32),
                                     "1.conv": StateCacheSpec((3, 2 * 20 + 56), torch.float32)}
    assert layout[2] == layout[0] and layout[1] == PagedCacheSpec(2, 12, 0, None, v_heads=2, v_head_dim=20)
    assert dict(layout[3].extra) == {"1.state": StateCacheSpec((3, 7, 5), torch.float32)}            # one tap keeps nothing
    assert model.graph_safe
    # equal constants share one table
    _, model = build(config([attention(), attention(), attention(temp=(0.3, 8))]))
    t = [b.mixer.query_temperature for b in model.blocks]
    assert t[0] is t[1] and t[0] is not t[2]


def test_key_heads_left_out_are_as_many_as_heads():
    raw = json.loads(json.dumps(CASES["A"]))
    for m in (raw["layers"][3]["mixer"]["left"], raw["layers"][3]["mixer"]["right"]):
        del m["kv_heads"]
    cfg, model = build(raw)
    assert model.blocks[2].mixer.members[0].kv_heads == 2 and model.blocks[2].mixer.members[1].kv_heads == 3


def test_random_model_folder_is_read_back_by_name(tmp_path):
    from carbon_engine_b200.weights.loader import check_tensors
    from carbon_engine_b200.weights.safetensors_io import TensorDirectory
    folder = write_model(CASES["A"], str(tmp_path / "A"))
    cfg, model = build(json.load(open(f"{folder}/config.json")))
    check_tensors(model.all_tensor_specs(), TensorDirectory(folder), model.all_ignorable_tensors())
    cfg2, w = plain.read_model(folder)
    assert cfg2["layers"][2]["weights_of"] == 0 and "l2.norm1" not in w and w["l0.mix.left.sink"].shape == (4,)


def test_sketch_config_shares_weights_on_request():
    from carbon_engine_b200.config.lanirax import sketch_config
    cfg = sketch_config(200, 64, 6, 4, 2, 16, 128, shared_from=4)
    assert [l["type"] for l in cfg.layers] == ["parallel", "attention"] * 3
    assert [l.get("weights_of") for l in cfg.layers] == [None] * 4 + [0, 1]
    _, model = build(cfg.to_json_dict())
    assert len(model.blocks) == 4 and len(model.schedule) == 6


def test_tables_of_the_package_against_the_plain_formulas():
    from carbon_engine_b200.models.lanirax import distance_slopes
    for name in ("A", "B", "C", "T", "V"):
        cfg, model = build(CASES[name], 200)
        for call, layer in zip(model.schedule, CASES[name]["layers"]):
            mixer, m = model.blocks[call.block].mixer, layer["mixer"]
            if layer["type"] == "attention":
                assert mixer.distance_slopes == distance_slopes(m["heads"])
                assert torch.allclose(torch.tensor(mixer.distance_slopes), torch.tensor(plain.distance_slopes(m["heads"])), rtol=1e-12)
                if m.get("q_temp"):
                    mixer.query_temperature.prepare(torch.device("cpu"))
                    want = plain.query_temperature(200, m["q_temp"]["coef"], m["q_temp"]["every"]).float()
                    assert torch.equal(mixer.query_temperature.table, want)
                continue
            pos, rot = mixer.members[0].position, m["left"].get("rot")
            if rot is None:
                assert pos is None
                continue
            pos.prepare(torch.device("cpu"))
            assert pos.pairing == "interleaved"
            freqs, amp = plain.stretched_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
            ang = torch.arange(200, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
            assert torch.allclose(pos.cos, (ang.cos() * amp).float(), atol=1e-6) and torch.allclose(pos.sin, (ang.sin() * amp).float(), atol=1e-6)


# ---- the plain implementation against hand-computed rows ------------------------------------------------------------
F = torch.float64


def test_plain_stretched_frequencies_by_hand():
    # dims 8, base 16: frequencies 1, 1/2, 1/4, 1/8.  original = 2 pi 64: the pair that turns t times is 8 ln(64 / t) / (2 ln 16):
    # t = 64 -> 0, t = 4 -> 4; so the ramp over the pairs 0..3 is 0, 1/4, 1/2, 3/4
    freqs, amp = plain.stretched_frequencies(8, 16.0, {"factor": 2.0, "original": 2 * math.pi * 64, "fast": 64.0 * (1 - 1e-12), "slow": 4.0 * (1 + 1e-12)})
    want = [f / 2 * r + f * (1 - r) for f, r in zip((1, 0.5, 0.25, 0.125), (0, 0.25, 0.5, 0.75))]
    assert freqs == pytest.approx(want, rel=1e-12) and amp == pytest.approx(1 + 0.1 * math.log(2.0))
    # a ramp of no width: every pair from its place on is divided
    freqs, _ = plain.stretched_frequencies(4, 100.0, {"factor": 5.0, "original": 1.0, "fast": 9.0, "slow": 9.0})
    assert freqs == pytest.approx([1.0, 0.1 / 5.0])
    assert plain.stretched_frequencies(4, 100.0, None) == ([1.0, 0.1], 1.0)
    x = torch.tensor([[[9.0, 9.0, 9.0]], [[1.0, 5.0, 7.0]]], dtype=F)
    r = plain.rotate_neighbours(x, {"dims": 2, "base": 10.0})
    assert torch.equal(r[0], x[0]) and float(r[1, 0, 2]) == 7.0
    assert torch.allclose(r[1, 0, :2], torch.tensor([math.cos(1) - 5 * math.sin(1), 5 * math.cos(1) + math.sin(1)], dtype=F))


def test_plain_temperature_slopes_window_and_sink_by_hand():
    t = plain.query_temperature(7, 0.5, 3)
    assert t.tolist() == pytest.approx([1, 1, 1 + 0.5 * math.log(2)] + [1 + 0.5 * math.log(2)] * 2 + [1 + 0.5 * math.log(3)] * 2)
    assert plain.distance_slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    q = k = torch.zeros(3, 1, 2, dtype=F)                   # all scores 0
    v = torch.tensor([[[2.0]], [[4.0]], [[12.0]]], dtype=F)
    run = lambda **kw: plain.softmax_attention(q, k, v, 1.0, **kw)[:, 0, 0]
    assert torch.allclose(run(), torch.tensor([2.0, 3.0, 6.0], dtype=F))
    assert torch.allclose(run(window=2), torch.tensor([2.0, 3.0, 8.0], dtype=F))
    assert torch.allclose(run(window=1), torch.tensor([2.0, 4.0, 12.0], dtype=F))
    assert torch.allclose(run(window=2, sink=torch.zeros(1, dtype=F)), torch.tensor([1.0, 2.0, 16 / 3], dtype=F))
    ln2 = math.log(2.0)                                     # a slope of ln 2 halves the weight per token of distance
    assert torch.allclose(run(slopes=[ln2]), torch.tensor([2.0, (1 + 4) / 1.5, (0.5 + 2 + 12) / 1.75], dtype=F))


def test_plain_recurrence_and_convolution_by_hand():
    q = torch.tensor([[1.0, 0.0]] * 3, dtype=F)
    v = torch.tensor([[3.0], [5.0], [7.0]], dtype=F)
    one = torch.ones(3, dtype=F)
    # beta 1, decay 1: a key written twice is overwritten, and the read-out sees the token's own write
    assert plain.delta_walk(q, q, v, one, one)[:, 0].tolist() == [3.0, 5.0, 7.0]
    other = torch.tensor([[1.0, 0.0], [0.0, 1.0], [0.0, 1.0]], dtype=F)
    assert plain.delta_walk(q, other, v, 0.5 * one, one)[:, 0].tolist() == [3.0, 1.5, 0.75]
    # the decay comes before the difference: u = beta (v - g S^T k)
    assert plain.delta_walk(q, q, v, 0.5 * one, 0.5 * one)[:, 0].tolist() == [1.5, 0.75 + 0.5 * (5 - 0.75), 1.4375 + 0.5 * (7 - 1.4375)]
    y = plain.short_convolution(torch.tensor([[1.0], [2.0], [3.0]], dtype=F), torch.tensor([[100.0, 10.0, 1.0]], dtype=F))
    assert y[:, 0].tolist() == [1.0, 12.0, 123.0]


def test_plain_mixture_by_hand():
    w = {"m.router": torch.tensor([[1.0], [2.0], [0.0]], dtype=F), "m.router.b": torch.tensor([0.0, 0.0, 1.5], dtype=F)}
    for e in range(3):
        for n in ("gate", "up", "down"):
            w[f"m.e{e}.{n}"] = torch.full((1, 1), float(e + 1), dtype=F)
    mlp = {"router": {"experts": 3, "top": 2}}
    margins = []
    got = plain.mixture(w, "m", mlp, torch.tensor([[1.0]], dtype=F), margins)          # logits 1, 2, 1.5: experts 1 and 2
    silu = lambda z: z / (1 + math.exp(-z))
    a, b = math.exp(2.0), math.exp(1.5)
    assert float(got) == pytest.approx((a * 2 * silu(2.0) * 2.0 + b * 3 * silu(3.0) * 3.0) / (a + b)) and margins == [[0.5]]


def test_plain_shared_layer_and_its_own_state(tmp_path):
    layer = pair(mlp=moe())
    folder = write_model(config([layer, shared(layer, 0)]), str(tmp_path / "m"))
    cfg, w = plain.read_model(folder)
    trace, first = [], []
    plain.forward(cfg, w, [3, 9, 27, 1], trace)
    plain.forward(dict(cfg, layers=cfg["layers"][:1]), w, [3, 9, 27, 1], first)
    assert torch.equal(trace[0], first[0]) and not torch.allclose(trace[1], trace[0])


def test_every_mechanism_moves_the_cases_logits(tmp_path):
    """What the configurations of the GPU tests are compared on must depend on every option: the plain model without it differs."""
    folder = write_model(CASES["A"], str(tmp_path / "A"), seed=11)
    cfg, w = plain.read_model(folder)
    toks = [int(t) for t in torch.randint(0, 97, (60,), generator=torch.Generator().manual_seed(1))]
    want = plain.forward(cfg, w, toks)

    def moved(change_cfg=None, change_w=None):
        c, t = json.loads(json.dumps(cfg)), dict(w)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(t)
        return float((plain.forward(c, t, toks) - want).abs().max() / want.abs().max())
    left = lambda c: c["layers"][0]["mixer"]["left"]
    assert moved(lambda c: left(c)["mask"].update(size=10)) > 1e-2
    assert moved(lambda c: left(c)["rot"]["scaling"].update(factor=4.0)) > 1e-3
    assert moved(lambda c: left(c)["rot"].pop("scaling")) > 1e-2
    assert moved(lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=8)) > 1e-4
    assert moved(lambda c: c.update(postln_alpha=1.2)) > 1e-2
    assert moved(None, lambda t: t.update({"l0.mix.left.sink": t["l0.mix.left.sink"] * 0 - 50})) > 1e-2
    assert moved(None, lambda t: t.update({"l0.mlp.router.b": t["l0.mlp.router.b"] * 0})) > 1e-3
    assert moved(None, lambda t: t.update({"embed.norm": t["embed.norm"] * 0 + 1})) > 1e-2
