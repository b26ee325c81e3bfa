"""Zoporax on the host: configuration and plan, tensor names, cache and state needs, the random-weights folder, and
the plain implementation's own mechanisms against independent closed forms."""
import copy
import json
import math

import numpy as np
import pytest

import helpers
import plain_zoporax as P

RAW = {"architecture": "Zoporax", "width": 40, "vocab": 70, "norm": {"eps": 1e-5},
       "layers": [
           {"type": "latent_attention",
            "mixer": {"heads": 3, "dim": 10, "rot_dim": 6, "vdim": 14, "kv_rank": 20, "q_rank": 12, "scale": 0.3, "mask": {"size": 9},
                      "rot": {"base": 300.0, "dims": 6, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}},
            "mlp": {"kind": "dense", "ff": 56}},
           {"type": "lightning", "mixer": {"heads": 2, "dim": 4, "vdim": 10, "decay": [0.5, 0.96875]},
            "mlp": {"kind": "moe", "expert": {"ff": 12}, "router": {"experts": 6, "top": 2, "scale": 1.7, "groups": {"count": 3, "keep": 2}},
                    "shared": {"ff": 20}}},
           {"type": "latent_attention",
            "mixer": {"heads": 2, "dim": 5, "rot_dim": 8, "vdim": 7, "kv_rank": 11, "q_rank": 9, "rot": {"base": 1000.0, "dims": 4}, "scale": 0.2},
            "mlp": None},
           {"type": "lightning", "mixer": {"heads": 1, "dim": 3, "vdim": 5, "decay": [1.0]},
            "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 3, "top": 3}}},
       ]}


def plan_of(raw):
    import cajeta_llm_b200  # noqa: F401
    from cajeta_llm_b200.config import parse_config_dict
    from cajeta_llm_b200.config.base import get_architecture
    cfg = parse_config_dict(raw)
    return cfg, get_architecture(cfg.architecture).build_plan(cfg)


def test_the_plan_follows_the_list_of_layers():
    cfg, plan = plan_of(RAW)
    assert [l.block.kind for l in plan.layers] == ["prenorm"] * 4
    assert [l.mixer.kind for l in plan.layers] == ["latent_attention", "lightning"] * 2
    assert [None if l.feed_forward is None else l.feed_forward.kind for l in plan.layers] == ["dense_gated", "sparse_moe", None, "sparse_moe"]
    assert [(e.layer, e.cache_from) for e in plan.schedule] == [(i, None) for i in range(4)]
    assert plan.lm_head_name is None and plan.embedding_name == "embed" and plan.final_norm.kind == "rmsnorm"
    lat = plan.layers[0].mixer
    assert (lat["q_rank"], lat["kv_rank"], lat["rot_dim"], lat["gate"], lat["window"], lat["halves"]) == (12, 20, 6, "entries", 9, True)
    assert lat["position"].kind == "rope" and lat["position"]["rotary_dim"] == 6 and lat["position"]["scaling"]["factor"] == 3.0
    assert plan.layers[2].mixer["window"] == 0 and plan.layers[2].mixer["position"]["scaling"] is None
    assert plan.layers[1].mixer["decay"] == (0.5, 0.96875)
    ff = plan.layers[1].feed_forward
    assert (ff["top_k"], ff["route_scale"], ff["route_groups"], ff["group_score"], ff["shared_intermediate_size"]) == (2, 1.7, (3, 2), "top2", 20)
    assert ff["activation"] == "gelu" and ff["score"] == "sigmoid" and ff["norm_topk_prob"] and ff["shared_gate"]
    bare = plan.layers[3].feed_forward
    assert (bare["route_scale"], bare["route_groups"], bare["shared_intermediate_size"], bare["shared_gate"]) == (1.0, None, 0, False)
    assert cfg.to_json_dict() == RAW


def test_tensor_names_shapes_and_needs():
    from cajeta_llm_b200.engine.model import build_model
    from cajeta_llm_b200.parts.base import Runtime
    cfg, _ = plan_of(RAW)
    model = build_model(cfg, Runtime("float32", "cpu"))
    specs = model.params()
    p = {n: tuple(s.shape) for n, s in specs.items()}
    assert p["l0.norm1"] == p["l0.norm2"] == p["final.norm"] == (40,)
    assert specs["l2.norm2"].optional and not specs["l0.norm2"].optional      # a layer without a feed-forward: nothing reads its norm
    assert p["l0.mix.dq"] == (12, 40) and p["l0.mix.dq.norm"] == (12,) and p["l0.mix.uq"] == (3 * 16, 12)
    assert p["l0.mix.dkv"] == (26, 40) and p["l0.mix.dkv.norm"] == (20,) and p["l0.mix.uk"] == (30, 20) and p["l0.mix.uv"] == (42, 20)
    assert p["l0.mix.g"] == (42, 40) and p["l0.mix.o"] == (40, 42) and "l0.mix.q" not in p and "l0.mix.sink" not in p
    assert p["l1.mix.q"] == p["l1.mix.k"] == (8, 40) and p["l1.mix.v"] == p["l1.mix.g"] == (20, 40) and p["l1.mix.norm"] == (20,)
    assert p["l1.mix.o"] == (40, 20)
    assert p["l0.mlp.gate"] == p["l0.mlp.up"] == (56, 40) and p["l0.mlp.gate.b"] == p["l0.mlp.up.b"] == (56,) and p["l0.mlp.down.b"] == (40,)
    assert p["l1.mlp.router"] == (6, 40) and p["l1.mlp.e5.up"] == (12, 40) and p["l1.mlp.e5.down"] == (40, 12) and "l1.mlp.e5.gate" not in p
    assert p["l1.mlp.shared.up"] == (20, 40) and p["l1.mlp.shared.down"] == (40, 20) and p["l1.mlp.shared.sg"] == (1, 40)
    assert "l1.mlp.shared.gate" not in p and "l3.mlp.shared.up" not in p and not any(n.startswith("l2.mlp") for n in p)
    assert p["embed"] == (70, 40) and "head" not in p
    kv = model.kv_needs()
    assert (kv[0].kv_heads, kv[0].head_dim, kv[0].values, kv[0].window) == (1, 26, False, 9)
    assert (kv[2].head_dim, kv[2].window) == (19, 0) and kv[1] is None and kv[3] is None
    st = model.state_needs()
    assert st[0] is None and st[2] is None and st[1].shape == (2 * 4 * 10,) and st[3].shape == (15,)


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="attention"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), "base"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("original"), "original"),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "kept groups"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "ff"),
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


def test_random_weights_folder_round_trip(tmp_path):
    helpers.write_model(str(tmp_path), RAW, seed=3)
    cfg, W = P.load_folder(str(tmp_path))
    assert cfg == RAW and W["l1.mix.norm"].shape == (20,) and "l2.norm2" not in W
    after = []
    logits = P.forward(cfg, W, [1, 2, 3, 4, 5], layer_outputs=after)
    assert logits.shape == (5, 70) and len(after) == 4 and after[0].shape == (5, 40) and bool(np.isfinite(logits).all())


def test_the_engine_s_frequency_table_equals_the_plain_one():
    from cajeta_llm_b200.parts.base import Runtime, make_part
    from cajeta_llm_b200.parts.plan import PartSpec
    for base, dims, scaling in ((300.0, 6, None), (500000.0, 24, {"factor": 3.0, "original": 512, "fast": 16.0, "slow": 2.0}),
                                (10000.0, 16, {"factor": 8.0, "original": 64, "fast": 32.0, "slow": 1.0})):
        part = make_part("position", PartSpec("rope", {"head_dim": dims, "rotary_dim": dims, "theta": base, "float64_table": True, "scaling": scaling}),
                         "", Runtime("float32", "cpu"))
        want, magnitude = P.frequencies({"base": base, "dims": dims, "scaling": scaling})
        assert np.allclose(part.inv_freq.double().numpy(), want, rtol=1e-7) and math.isclose(part.magnitude, magnitude)


def test_the_lightning_part_s_tables():
    from cajeta_llm_b200.csrc import kernels as K
    from cajeta_llm_b200.parts.base import Runtime, make_part
    from cajeta_llm_b200.parts.plan import PartSpec
    spec = {"hidden_size": 8, "heads": 3, "dim": 4, "vdim": 6, "decay": (0.0, 0.75, 1.0), "eps": 1e-6}
    part = make_part("mixer", PartSpec("lightning", spec), "m", Runtime("bfloat16", "cpu"))
    assert part.powers.shape == (3, K.DECAY_CHUNK + 1)
    assert part.powers[0].tolist() == [1.0] + [0.0] * K.DECAY_CHUNK and part.powers[2].tolist() == [1.0] * (K.DECAY_CHUNK + 1)
    assert math.isclose(float(part.powers[1, 64]), 0.75 ** 64, rel_tol=1e-6)
    assert part.log2_decay.tolist()[0] == -math.inf and part.log2_decay.tolist()[2] == 0.0
    for bad in ((0.5, 0.5), (0.5, 0.5, -0.1), (0.5, 0.5, 1.01)):
        with pytest.raises(ValueError):
            make_part("mixer", PartSpec("lightning", dict(spec, decay=bad)), "m", Runtime("float32", "cpu"))


def test_rotation_pairs_halves_and_keeps_relative_angles():
    rng = np.random.default_rng(0)
    a, b = rng.normal(size=10), rng.normal(size=10)
    rot = {"base": 100.0, "dims": 6}
    d1 = P.rotate_halves(a, 17, rot) @ P.rotate_halves(b, 12, rot)
    d2 = P.rotate_halves(a, 105, rot) @ P.rotate_halves(b, 100, rot)
    assert abs(d1 - d2) < 1e-9
    assert np.array_equal(P.rotate_halves(a, 9, rot)[6:], a[6:])
    one = P.rotate_halves(np.array([1.0, 0.0, 0.0, 0.0]), 3, {"base": 100.0, "dims": 4})
    assert np.allclose(one, [math.cos(3.0), 0.0, math.sin(3.0), 0.0])
    # stretched: the fastest frequency stays, the slowest is divided by the factor, lengths grow by the magnitude
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    f, m = P.frequencies(rot)
    assert f[0] == 1.0 and math.isclose(f[15], 10000.0 ** (-30 / 32) / 4.0) and math.isclose(m, 1.0 + 0.1 * math.log(4.0))
    v = rng.normal(size=32)
    assert math.isclose(np.linalg.norm(P.rotate_halves(v, 77, rot)), m * np.linalg.norm(v))


def test_the_window_counts_the_row_itself():
    assert [P.first_visible(t, {"size": 3}) for t in (0, 1, 2, 3, 10)] == [0, 0, 0, 1, 8]
    assert P.first_visible(10, None) == 0 and P.first_visible(10, {"size": 1}) == 10


def test_gelu_in_both_forms():
    assert math.isclose(P.gelu_erf(np.array([1.0]))[0], 0.8413447460685429)
    z = np.linspace(-6, 6, 50)
    assert np.abs(P.gelu_erf(z) - P.gelu_tanh(z)).max() < 1e-3 and np.abs(P.gelu_erf(z) - P.gelu_tanh(z)).max() > 1e-4
    # as a gate: z sigmoid(alpha z + cubic z^3)
    from cajeta_llm_b200.csrc.kernels import GELU_TANH
    assert np.allclose(P.gelu_tanh(z), z * P.sigmoid(GELU_TANH[0] * z + GELU_TANH[1] * z ** 3))


def test_linear_attention_by_hand():
    """One head, dim 1, vdim 2, two tokens: the state and the read-out written out."""
    m = {"heads": 1, "dim": 1, "vdim": 2, "decay": [0.5]}
    W = {".q": np.array([[1.0]]), ".k": np.array([[2.0]]), ".v": np.array([[1.0], [-1.0]]), ".g": np.zeros((2, 1)), ".o": np.eye(2), ".norm": np.array([2.0, 4.0])}
    h = np.array([[1.0], [0.5]])
    s = lambda z: z / (1.0 + math.exp(-z))
    S0 = s(2.0) * np.array([s(1.0), s(-1.0)])
    S1 = 0.5 * S0 + s(1.0) * np.array([s(0.5), s(-0.5)])
    got = P.lightning(h, W, "", m, 1e-6)
    for row, S, q in ((0, S0, s(1.0)), (1, S1, s(0.5))):
        o = S * q
        assert np.allclose(got[row], o / math.sqrt(np.mean(o * o) + 1e-6) * np.array([2.0, 4.0]) * 0.5)
    # a state handed over is the same as one sequence
    state = np.zeros((1, 1, 2))
    first = P.lightning(h[:1], W, "", m, 1e-6, state)
    assert np.allclose(np.concatenate([first, P.lightning(h[1:], W, "", m, 1e-6, state)]), got)


def test_the_router_keeps_groups_by_their_two_best_scores():
    scores = np.array([0.9, 0.1, 0.1, 0.6, 0.5, 0.1, 0.8, 0.0, 0.2])          # pairs: 1.0, 1.1, 1.0
    assert P.kept_experts(scores, {"count": 3, "keep": 1}) == [3, 4, 5]
    assert P.kept_experts(scores, {"count": 3, "keep": 2}) == [0, 1, 2, 3, 4, 5]
    assert P.kept_experts(scores[:3], {"count": 3, "keep": 2}) == [0, 1]      # groups of one: their only score
    z = np.log(scores[:6] / (1.0 - scores[:6]))
    W = {".router": np.diag(z)}
    ff = {"router": {"experts": 6, "top": 2, "scale": 3.0, "groups": {"count": 2, "keep": 1}}}
    picks, weights = P.route(np.ones((1, 6)), W, "", ff)
    assert picks == [[3, 4]] and np.allclose(weights, [[3.0 * 0.6 / 1.1, 3.0 * 0.5 / 1.1]])


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
    assert config == RAW and W["l1.mlp.e5.down"].shape == (40, 12) and W["l0.mlp.down.b"].shape == (40,)
