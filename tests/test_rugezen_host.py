"""Rugezen on the host: configuration and plan, tensor names, cache and state needs, the random-weights folder, and the
plain implementation's own mechanisms against independent closed forms."""
import copy
import json
import math

import numpy as np
import pytest

import helpers
import plain_rugezen as P

RAW = {"architecture": "Rugezen", "width": 40, "vocab": 70, "norm": {"eps": 1e-4}, "residual_mult": 0.37,
       "loop": {"start": 1, "stop": 3, "times": 3},
       "layers": [
           {"type": "mingru", "mixer": {"width": 26}, "mlp": None},
           {"type": "attention",
            "mixer": {"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 14, "rot": {"base": 300.0, "dims": 4}, "scale": 0.3, "softcap": 12.0},
            "mlp": {"kind": "dense", "ff": 56}},
           {"type": "mingru", "mixer": {"width": 64}, "mlp": {"kind": "dense", "ff": 20}},
           {"type": "attention",
            "mixer": {"heads": 3, "kv_heads": 3, "dim": 8, "vdim": 5, "rot": {"base": 10000.0, "dims": 8}, "scale": 0.5, "softcap": 40.0},
            "mlp": None},
       ]}


def plan_of(raw):
    import cajeta_llm_b200  # noqa: F401
    from cajeta_llm_b200.config import parse_config_dict
    from cajeta_llm_b200.config.base import get_architecture
    cfg = parse_config_dict(raw)
    return cfg, get_architecture(cfg.architecture).build_plan(cfg)


def test_the_plan_follows_the_list_of_layers_and_the_loop():
    cfg, plan = plan_of(RAW)
    assert [l.block.kind for l in plan.layers] == ["parallel"] * 4 and all(l.block["residual_mult"] == 0.37 for l in plan.layers)
    assert [l.mixer.kind for l in plan.layers] == ["mingru", "attention", "mingru", "attention"]
    assert [None if l.feed_forward is None else l.feed_forward.kind for l in plan.layers] == [None, "dense_relu2", "dense_relu2", None]
    assert [e.layer for e in plan.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert all(e.cache_from is None and e.before is None for e in plan.schedule)
    att = plan.layers[1].mixer
    assert (att["num_heads"], att["num_kv_heads"], att["head_dim"], att["value_dim"], att["scale"], att["softcap"]) == (6, 2, 10, 14, 0.3, 12.0)
    assert att["sink_score"] == 0.0 and att["qk_norm"] == {"eps": 1e-4} and att["value_norm"] == {"eps": 1e-4}
    assert att["position"]["pairs"] and att["position"]["rotary_dim"] == 4 and att["position"]["theta"] == 300.0
    assert plan.layers[2].feed_forward["bias"] and plan.lm_head_name == "head"
    assert cfg.to_json_dict() == RAW
    bare = {k: v for k, v in RAW.items() if k != "loop"}
    cfg2, plan2 = plan_of(bare)
    assert [e.layer for e in plan2.schedule] == [0, 1, 2, 3] and cfg2.to_json_dict() == bare


def test_tensor_names_shapes_and_needs():
    from cajeta_llm_b200.engine.model import build_model
    from cajeta_llm_b200.parts.base import Runtime
    cfg, _ = plan_of(RAW)
    model = build_model(cfg, Runtime("float32", "cpu"))
    p = {n: tuple(s.shape) for n, s in model.params().items() if not s.optional}
    assert p == {
        "embed": (70, 40), "head": (70, 40), "final.norm": (40,),
        "l0.norm1": (40,), "l0.mix.z": (26, 40), "l0.mix.z.b": (26,), "l0.mix.x": (26, 40), "l0.mix.x.b": (26,), "l0.mix.g": (26, 40), "l0.mix.o": (40, 26),
        "l1.norm1": (40,), "l1.norm2": (40,), "l1.mix.q": (60, 40), "l1.mix.k": (20, 40), "l1.mix.v": (28, 40), "l1.mix.o": (40, 84),
        "l1.mlp.up": (56, 40), "l1.mlp.up.b": (56,), "l1.mlp.down": (40, 56), "l1.mlp.down.b": (40,),
        "l2.norm1": (40,), "l2.norm2": (40,), "l2.mix.z": (64, 40), "l2.mix.z.b": (64,), "l2.mix.x": (64, 40), "l2.mix.x.b": (64,), "l2.mix.g": (64, 40),
        "l2.mix.o": (40, 64), "l2.mlp.up": (20, 40), "l2.mlp.up.b": (20,), "l2.mlp.down": (40, 20), "l2.mlp.down.b": (40,),
        "l3.norm1": (40,), "l3.mix.q": (24, 40), "l3.mix.k": (24, 40), "l3.mix.v": (15, 40), "l3.mix.o": (40, 15)}
    assert {n for n, s in model.params().items() if s.optional} == {"l0.norm2", "l3.norm2"}
    # every pass over the looped stretch has a cache or a state of its own
    kv, st = model.kv_needs(), model.state_needs()
    assert [None if k is None else (k.kv_heads, k.head_dim, k.value_dim, k.window) for k in kv] == \
        [None, (2, 10, 14, 0), None, (2, 10, 14, 0), None, (2, 10, 14, 0), None, (3, 8, 5, 0)]
    assert [None if s is None else s.shape for s in st] == [(26,), None, (64,), None, (64,), None, (64,), None]


def test_the_residual_multiplier_reaches_both_sublayers():
    from cajeta_llm_b200.engine.model import build_model
    from cajeta_llm_b200.parts.base import Runtime
    cfg, _ = plan_of(RAW)
    model = build_model(cfg, Runtime("float32", "cpu"))
    assert all(b.mixer.out_scale == 0.37 and (b.feed_forward is None or b.feed_forward.out_scale == 0.37) for b in model.blocks)
    from cajeta_llm_b200.parts.base import make_part
    from cajeta_llm_b200.parts.plan import LayerSpec, PartSpec
    norm = PartSpec("rmsnorm", {"dim": 8, "eps": 1e-5, "weight_name": ""})
    block = PartSpec("parallel", {"mixer_norm_name": "a", "feed_forward_norm_name": "b", "mixer_name": "m", "feed_forward_name": "f", "residual_mult": 0.5})
    layer = LayerSpec(prefix="l0", block=block, mixer=PartSpec("mingru", {"hidden_size": 8, "width": 4}),
                      feed_forward=PartSpec("dense_swiglu", {"hidden_size": 8, "intermediate_size": 4}), mixer_norm=norm, feed_forward_norm=norm)
    with pytest.raises(ValueError, match="out_scale"):
        make_part("block", block, "l0", Runtime("float32", "cpu"), layer=layer)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="gru"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(width=0), "width"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=3), "dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][1]["mlp"].update(ff=0), "ff"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.update(residual_mult="half"), "residual_mult"),
    (lambda c: c.pop("norm"), "norm.eps"),
    (lambda c: c.pop("layers"), "layers"),
])
def test_configuration_errors_name_the_key(change, message):
    from cajeta_llm_b200.config.base import ConfigError
    raw = copy.deepcopy(RAW)
    change(raw)
    with pytest.raises(ConfigError) as e:
        plan_of(raw)
    assert message in str(e.value)


def test_attention_options_that_do_not_go_together_are_refused():
    from cajeta_llm_b200.parts.base import Runtime, make_part
    from cajeta_llm_b200.parts.plan import PartSpec
    base = {"hidden_size": 32, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "position": PartSpec("none")}
    rt = Runtime("float32", "cpu")
    for extra in ({"qk_norm": {"eps": 1e-5}, "value_norm": {"eps": 1e-6}}, {"values_from_keys": True, "value_norm": {"eps": 1e-5}},
                  {"sink_score": 0.0, "talk": "t"}, {"value_norm": {"eps": 1e-5}, "sink": "s"}, {"sink_score": 0.0, "qkv_bias": True}):
        with pytest.raises(ValueError):
            make_part("mixer", PartSpec("attention", dict(base, **extra)), "m", rt)
    part = make_part("mixer", PartSpec("attention", dict(base, qk_norm={"eps": 1e-5}, scale=0.25)), "m", rt)
    assert part.unit_qk and 2.0 < part.score_bound < 2.1 and part.params().keys() == {"m.q_proj.weight", "m.k_proj.weight", "m.v_proj.weight", "m.o_proj.weight"}


def test_random_weights_folder_round_trip(tmp_path):
    helpers.write_model(str(tmp_path), RAW, seed=3)
    cfg, W = P.load_folder(str(tmp_path))
    assert cfg == RAW and W["l1.mix.q"].shape == (60, 40) and "l0.norm2" not in W and "l3.norm2" not in W
    after = []
    logits = P.forward(cfg, W, [1, 2, 3, 4, 5], layer_outputs=after)
    assert logits.shape == (5, 70) and len(after) == 8 and after[0].shape == (5, 40) and bool(np.isfinite(logits).all())


def test_the_frequency_table_is_rounded_once():
    from cajeta_llm_b200.parts.base import Runtime, make_part
    from cajeta_llm_b200.parts.plan import PartSpec
    for base, dims in ((300.0, 4), (500000.0, 32), (10000.0, 16)):
        part = make_part("position", PartSpec("rope", {"head_dim": dims, "rotary_dim": dims, "theta": base, "pairs": True, "float64_table": True}), "",
                         Runtime("float32", "cpu"))
        want = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64).astype(np.float32)
        assert np.array_equal(part.inv_freq.numpy(), want) and part.pairs


def test_rotation_keeps_a_head_s_length_so_the_norm_may_come_first():
    rng = np.random.default_rng(0)
    v = rng.normal(size=10)
    r = P.rotate_pairs(v, 23, 100.0, 6)
    assert math.isclose(np.dot(v, v), np.dot(r, r)) and np.array_equal(r[6:], v[6:])
    assert np.allclose(P.unit_rms(r, 1e-3), P.rotate_pairs(P.unit_rms(v, 1e-3), 23, 100.0, 6))
    assert np.allclose(P.rotate_pairs(np.array([1.0, 0.0, 0.0, 1.0]), 3, 100.0, 4), [math.cos(3.0), math.sin(3.0), -math.sin(0.3), math.cos(0.3)])


def test_the_divisor_is_one_larger_than_the_sum_of_the_keys():
    s = np.array([0.3, -1.0, 2.0])
    e = np.exp(s)
    assert np.allclose(P.softmax_plus_one(s), e / (1.0 + e.sum()))
    assert np.allclose(P.softmax_plus_one(s - 800.0), 0.0) and np.allclose(P.softmax_plus_one(s + 800.0), e / e.sum())


def test_attention_by_hand():
    """One head of two entries, no rotation, identity projections: the second row's two scores by hand."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.5, "softcap": 2.0}
    W = {".q": np.eye(2), ".k": np.array([[0.0, 1.0], [1.0, 0.0]]), ".v": 3.0 * np.eye(2), ".o": np.eye(2)}
    h = np.array([[3.0, 4.0], [1.0, 0.0]])
    got = P.attention(h, W, "", m, 0.0)
    r = math.sqrt(2.0)
    unit = np.array([[0.6 * r, 0.8 * r], [r, 0.0]])                    # rows over their root mean square; values alike, 3 cancels
    keys = unit[:, ::-1]
    s = 2.0 * np.tanh(1.5 * (keys @ unit[1]) / 2.0)
    want = (np.exp(s) @ unit) / (1.0 + np.exp(s).sum())
    assert np.allclose(got[1], want)
    s0 = 2.0 * math.tanh(1.5 * float(keys[0] @ unit[0]) / 2.0)
    assert np.allclose(got[0], unit[0] * math.exp(s0) / (1.0 + math.exp(s0)))


def test_the_recurrence_by_hand():
    """Gates and candidates at chosen values: a shut gate keeps the state, an open one replaces it, in between they mix."""
    W = {".z": np.array([[1.0, 0.0]]), ".z.b": np.array([0.0]), ".x": np.array([[0.0, 1.0]]), ".x.b": np.array([0.25]),
         ".g": np.array([[0.0, 0.0]]), ".o": np.array([[1.0], [2.0]])}
    h = np.array([[50.0, 1.75], [-50.0, 9.0], [0.0, -1.25], [50.0, -0.25]])
    W[".g"] = np.array([[0.02, 0.0]])
    got = P.min_gru(h, W, "")
    gate = P.silu(h[:, 0] * 0.02)
    S = [2.5, 2.5, 0.5 * 2.5 + 0.5 / (1.0 + math.e), 0.5]              # u = 2, 9.25 (kept out), -1, 0: its candidate one half
    assert np.allclose(got[:, 0], np.array(S) * gate) and np.allclose(got[:, 1], 2.0 * got[:, 0])
    assert math.isclose(float(P.candidate(np.array(-1e-9))), 0.5, rel_tol=1e-6) and float(P.candidate(np.array(0.0))) == 0.5


def test_stretches_of_the_recurrence_compose():
    """A stretch of tokens acts on the state as one map S -> A S + B; cut anywhere, the maps compose to the same result."""
    rng = np.random.default_rng(1)
    a, b, S0 = rng.uniform(size=20), rng.normal(size=20), 0.7
    S = S0
    for i in range(20):
        S = a[i] * S + b[i]

    def stretch(lo, hi):
        A, B = 1.0, 0.0
        for i in range(lo, hi):
            A, B = a[i] * A, a[i] * B + b[i]
        return A, B

    for cut in (1, 7, 19):
        (A1, B1), (A2, B2) = stretch(0, cut), stretch(cut, 20)
        assert math.isclose(A2 * (A1 * S0 + B1) + B2, S)
        assert math.isclose(A2 * A1 * S0 + (A2 * B1 + B2), S)


def test_the_feed_forward_squares_what_the_bias_lets_through():
    W = {".up": np.array([[1.0], [1.0]]), ".up.b": np.array([-1.0, 2.0]), ".down": np.array([[1.0, 10.0]]), ".down.b": np.array([0.5])}
    assert np.allclose(P.feed_forward(np.array([[3.0], [-4.0]]), W, ""), [[4.0 + 250.0 + 0.5], [0.5]])


def test_the_looped_layers_run_in_order():
    assert P.layer_order(RAW) == [0, 1, 2, 1, 2, 1, 2, 3]
    assert P.layer_order({"layers": [1, 2, 3]}) == [0, 1, 2]


def test_command_line_writes_a_random_model_folder(tmp_path):
    import subprocess
    import sys
    cfg = tmp_path / "config.json"
    cfg.write_text(json.dumps(RAW))
    out = tmp_path / "model"
    r = subprocess.run([sys.executable, "-m", "cajeta_llm_b200", "random-weights", "--config", str(cfg), "--seed", "4", "--out", str(out)],
                       cwd=helpers.ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-1000:]
    config, W = P.load_folder(str(out))
    assert config == RAW and W["l2.mix.z.b"].shape == (64,) and W["l2.mlp.down.b"].shape == (40,)
