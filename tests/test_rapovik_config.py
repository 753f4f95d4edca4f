"""What needs no GPU of the Rapovik design: reading its config.json, the order of the layer runs, the caches its blocks ask for,
tensor names, the order in which rows are held, and the plain implementation's own consistency."""
import json
import math
import os

import pytest
import torch

import plain_rapovik as plain
from rapovik_cases import CASES, SINGLE, attention, config, mamba, mlstm, moe, write_model


def test_config_round_trip_and_registry(tmp_path):
    from carbon_engine_b200.config.rapovik import RapovikConfig
    from carbon_engine_b200.config.registry import load_config
    for name, raw in list(CASES.items()) + list(SINGLE.items()):
        folder = write_model(raw, str(tmp_path / name))
        arch, cfg = load_config(folder)
        assert arch.name == "Rapovik" and cfg == RapovikConfig.from_dict(json.loads(json.dumps(raw)))
        with open(os.path.join(folder, "config.json")) as fh:
            assert RapovikConfig.from_dict(json.load(fh)) == cfg
        pcfg, w = plain.read_model(folder)
        assert pcfg["vocab"] == raw["vocab"] and w["embed"].shape == (raw["vocab"], raw["width"])
        assert list(cfg.layer_runs()) == plain.layer_runs(pcfg)
    assert RapovikConfig.from_dict(CASES["A"]).layer_runs() == (0, 1, 2, 1, 2, 3)
    assert RapovikConfig.from_dict(CASES["B"]).layer_runs() == (0, 1, 0, 1, 0, 1, 2, 3)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="conv"), "unknown layer type"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=64), "at most rot_dim"),
    (lambda c: c["layers"][2]["mixer"].update(mask={}), "size"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].update(groups=3), "multiple of 3 groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=7), "norm_groups=7"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mixer"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][1]["mlp"].update(kind="routed"), "dense"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "expert: 'limit'"),
    (lambda c: c["layers"][1]["mlp"]["shared"].pop("ff"), "shared: 'ff'"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top=9"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=0), "keep"),
    (lambda c: c["loop"].update(stop=9), "does not lie"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("width"), "width"),
])
def test_config_errors_name_the_key(change, message):
    from carbon_engine_b200.config.base import ConfigError
    from carbon_engine_b200.config.rapovik import RapovikConfig
    raw = json.loads(json.dumps(CASES["A"]))
    change(raw)
    with pytest.raises(ConfigError, match=message):
        RapovikConfig.from_dict(raw)


def _build(raw, positions=256):
    import carbon_engine_b200.models  # noqa: F401
    from carbon_engine_b200.config.rapovik import RapovikConfig
    from carbon_engine_b200.config.registry import resolve_architecture
    return resolve_architecture(raw).build_model(RapovikConfig.from_dict(raw), positions)


def test_schedule_caches_and_tensor_names():
    from carbon_engine_b200.parts.base import BundleCacheSpec, PagedCacheSpec, StateCacheSpec
    model = _build(CASES["A"])
    # every run of a looped layer has a cache of its own
    assert [(c.block, c.cache, c.writes) for c in model.schedule] == [(0, 0, True), (1, 1, True), (2, 2, True), (1, 3, True), (2, 4, True), (3, 5, True)]
    layout = dict(model.cache_layout())
    f32 = torch.float32
    assert layout[0] == BundleCacheSpec(StateCacheSpec((4, 12, 10), f32), (("conv", StateCacheSpec((3, 40 + 2 * 24), f32)),))
    assert layout[1] == layout[3] == BundleCacheSpec(StateCacheSpec((3, 8 * 13), f32), (("maximum", StateCacheSpec((3,), f32)),))
    assert layout[2] == layout[4] == PagedCacheSpec(1, 14 + 8, 21, None, v_heads=1, v_head_dim=0)
    shapes = {s.name: tuple(s.shape) for s in model.all_tensor_specs()}
    assert shapes["l0.mix.in"] == (2 * 40 + 2 * 24 + 4, 40) and shapes["l0.mix.conv"] == (88, 4) and shapes["l0.mix.conv.b"] == (88,)
    assert shapes["l0.mix.norm"] == (40,) and shapes["l1.mix.norm"] == (36,) and shapes["l1.mix.i"] == (3, 40) and shapes["l1.mix.f.b"] == (3,)
    assert shapes["l0.mlp.gate.b"] == (40,) and shapes["l0.mlp.down.b"] == (40,) and shapes["l1.mlp.correction"] == (6,)
    assert shapes["l2.mix.q"] == (3 * 20, 40) and shapes["l2.mix.dkv"] == (22, 40)
    names = set(shapes)
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.dt_bias", "l0.mix.A_log", "l0.mix.D",
            "l1.mlp.router", "l1.mlp.e5.gate", "l1.mlp.e5.up", "l1.mlp.e5.down", "l1.mlp.shared.gate"} <= names
    assert not any(n.endswith(".b") for n in names if ".e0." in n or ".shared." in n) and "l1.mlp.e6.up" not in names
    assert model.graph_safe
    b = {s.name for s in _build(CASES["B"]).all_tensor_specs()}
    assert "l0.norm2" not in b and "l0.norm2b" not in b and not any(n.startswith("l0.mlp") for n in b)        # no feed-forward, no norms of it
    assert not any(n.startswith("l2.mlp.shared") for n in b)
    assert dict(_build(CASES["B"]).cache_layout())[6] == StateCacheSpec((3, 5, 8), f32)       # one tap: nothing of the convolution is kept


def test_rows_are_held_in_the_order_the_kernels_read():
    """The state-space projection's stored rows z | x | B | C | dt are held as C | B | x | z | dt, its convolution's rows likewise;
    a gated expert's gate and up rows by turns."""
    model = _build(config([mamba(heads=2, vdim=3, state=5, groups=2, conv=2, mlp=moe(experts=2, top=1, ff=3, groups=None))], width=8))
    rows = {"l0.mix.in": 2 * 6 + 2 * 10 + 2, "l0.mix.conv": 26, "l0.mix.conv.b": 26}

    def get(name):
        spec = next(s for s in model.all_tensor_specs() if s.name == name)
        t = torch.zeros(spec.shape)
        if name in rows:
            t += torch.arange(float(rows[name])).reshape([-1] + [1] * (len(spec.shape) - 1))
        if ".gate" in name or ".up" in name:
            t += torch.arange(float(spec.shape[0]))[:, None] + (100.0 if ".up" in name else 0.0)
        return t
    model.load_weights(get, torch.device("cpu"), torch.float32)
    mix, ff = model.blocks[0].mixer, model.blocks[0].ffn
    z, x, b, c, dt = range(0, 6), range(6, 12), range(12, 22), range(22, 32), range(32, 34)
    assert mix.inp.weight[:34, 0].tolist() == [float(i) for r in (c, b, x, z, dt) for i in r]
    assert mix.conv_w[:, 1].tolist() == mix.conv_b.tolist() == [float(i - 6) for r in (c, b, x) for i in r]
    assert ff.up[1, :, 0].tolist() == [0.0, 100.0, 1.0, 101.0, 2.0, 102.0]


def test_cache_storage_has_a_state_for_every_run():
    from carbon_engine_b200.cache.storage import CacheStorage
    model = _build(CASES["A"], 128)
    st = CacheStorage(model, torch.float32, torch.device("cpu"), 8, 10, 3, 128)
    views = [st.view(c) for c in model.schedule]
    assert views[2].k_pool.shape == (10, 1, 8, 14 + 8) and views[2].k_pool.data_ptr() != views[4].k_pool.data_ptr()
    assert views[1].state.shape == (3, 3, 8 * 13) and views[1].state.data_ptr() != views[3].state.data_ptr()
    assert st.bytes_per_token() == 2 * (14 + 8) * 4
    for v in (views[0], views[1], views[3]):
        v.state.fill_(1.0)
        for t in v.extra.values():
            t.fill_(1.0)
    st.zero_state(1)                     # a slot that a new request takes starts from nothing in every run's state
    for v in (views[0], views[1], views[3]):
        for t in (v.state, *v.extra.values()):
            assert float(t[1].abs().max()) == 0.0 and float(t[0].min()) == 1.0


def test_plain_pieces_agree_with_themselves():
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64) * 0.5
    # the rotation turns neighbours: a rotation by the angle, lengths kept, the rest untouched
    x = rnd(5, 2, 8)
    y = plain.rotate_neighbours(x, torch.arange(5), 6, 30.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    a = 3.0 * 30.0 ** (-2.0 / 6)
    assert abs(float(y[3, 1, 2]) - float(x[3, 1, 2] * math.cos(a) - x[3, 1, 3] * math.sin(a))) < 1e-12
    assert abs(float(y[3, 1, 3]) - float(x[3, 1, 3] * math.cos(a) + x[3, 1, 2] * math.sin(a))) < 1e-12
    # the window: a row sees itself and the size - 1 tokens before it
    p = plain.window_softmax(torch.zeros(6, 6, dtype=torch.float64), 3)
    assert [int((r > 0).sum()) for r in p] == [1, 2, 3, 3, 3, 3] and float(p[4, 2]) == pytest.approx(1 / 3) and float(p[4, 1]) == 0.0
    # the state-space walk against its closed form
    T, N, dv = 6, 3, 2
    xs, B, C, dt = rnd(T, dv), rnd(T, N), rnd(T, N), torch.rand(T, generator=g, dtype=torch.float64)
    out = plain.state_space_walk(xs, B, C, dt, 0.7, 0.3)
    for t in range(T):
        want = 0.3 * xs[t]
        for j in range(t + 1):
            want = want + math.exp(-0.7 * float(dt[j + 1:t + 1].sum())) * dt[j] * float(B[j] @ C[t]) * xs[j]
        assert torch.allclose(out[t], want, atol=1e-12)
    # the matrix memory's running maximum only rescales: with log gates near 0 it equals the plain weighted sum
    q, k, v = rnd(T, N), rnd(T, N), rnd(T, dv)
    li, lf = rnd(T), plain.log_sigmoid(rnd(T))
    out = plain.matrix_memory_walk(q, k, v, li, lf)
    for t in range(T):
        w = [math.exp(float(li[j]) + float(lf[j + 1:t + 1].sum())) * float(k[j] @ q[t]) for j in range(t + 1)]
        num = sum(w[j] * v[j] for j in range(t + 1))
        m = 0.0
        for j in range(t + 1):
            m = max(float(lf[j]) + m, float(li[j]))
        want = num * math.exp(-m) / (max(abs(sum(w)) * math.exp(-m), math.exp(-m)) + 1e-6)
        assert torch.allclose(out[t], want, atol=1e-10)
    # the activation's clamps and the convolution's last tap
    y = plain.clamped_glu(torch.tensor([3.0, -9.0]), torch.tensor([-4.0, 0.25]), 2.0)
    assert float(y[0]) == pytest.approx(2.0 / (1 + math.exp(-3.404)) * -1.0) and float(y[1]) == pytest.approx(-9.0 / (1 + math.exp(1.702 * 9)) * 1.25)
    c = plain.causal_conv(torch.tensor([[1.0], [10.0]], dtype=torch.float64), torch.tensor([[2.0, 3.0]], dtype=torch.float64),
                          torch.tensor([0.5], dtype=torch.float64))
    assert c[:, 0].tolist() == [3.5, 32.5]


def test_plain_router():
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    logit = lambda s: torch.log(torch.tensor(s, dtype=torch.float64) / (1 - torch.tensor(s, dtype=torch.float64)))
    s = [0.9, 0.05, 0.5, 0.55, 0.3, 0.3]
    zero = torch.zeros(6, dtype=torch.float64)
    # a group wins by the SUM of its two largest, not by its largest
    chosen, weights = plain.route(logit(s), zero, r)
    assert chosen == [3, 2] and weights == pytest.approx([0.55, 0.5])                  # not renormalized
    # the correction moves the choice (down to negative choice scores) but not the weights
    corr = torch.tensor([0.0, 0.0, -2.0, -2.0, -1.0, -1.0], dtype=torch.float64)
    chosen, weights = plain.route(logit(s), corr, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert chosen == [0, 1] and weights == pytest.approx([0.9, 0.05])
    chosen, weights = plain.route(logit(s), corr - 1.0, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert chosen == [0, 1, 4] and weights == pytest.approx([0.9, 0.05, 0.3])          # -1.7 is chosen: a barred expert is not 0
    chosen, _ = plain.route(logit(s), zero, {"experts": 6, "top": 3})
    assert chosen == [0, 3, 2]


def test_sketch_config_and_random_weights(tmp_path):
    from carbon_engine_b200.config.rapovik import sketch_config
    from carbon_engine_b200.weights.loader import write_random_model
    cfg = sketch_config(vocab=90, width=48, n_layers=4, heads=3, head_dim=8, ff=64, experts=6, top=2, groups=(3, 2), window=9, loop=(1, 3, 2))
    assert [(l["type"], l["mlp"]["kind"]) for l in cfg.layers] == [("mamba2", "dense"), ("mlstm", "moe"), ("latent_attention", "moe"), ("mamba2", "moe")]
    folder = write_random_model(cfg, str(tmp_path / "m"), seed=4)
    pcfg, w = plain.read_model(folder)
    logits = plain.forward(pcfg, w, [1, 5, 7, 2])
    assert logits.shape == (4, 90) and bool(torch.isfinite(logits).all())
    assert abs(float(w["l0.norm1b"].mean())) < 0.2 and abs(float(w["l0.mix.norm"].mean()) - 1.0) < 0.2
    # a layer without a feed-forward and one of each mixer alone also run
    assert plain.forward(config([attention(), mlstm()]), plain.read_model(write_model(config([attention(), mlstm()]), str(tmp_path / "n")))[1],
                         [3, 4]).shape == (2, 97)
