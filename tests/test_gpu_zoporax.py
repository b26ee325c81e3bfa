"""Zoporax through the engine against the plain implementation (``plain_zoporax.py``), and its kernels against their formulas.

Small configurations of their own whose sizes differ in every field (values of another size than keys, ranks and head counts
that are neither 1 nor equal to one another, and some that are 1; a rotation over a part of the rotated entries, with and
without stretched frequencies; windows, no window, a window of one; decays of 0 and 1; layers without a feed-forward,
routers without groups, without a scale, with groups of one, without a shared expert).  Each mechanism alone as a small model; whole
prompts against token-by-token decoding and portions down to two tokens; unequal requests in one batch against each alone;
slots and pages used again; attention made sharp so that single keys - at page borders, just inside and just outside a window -
decide a row, in prompts and in decoding; memories that reach far back; first tokens; long decoding; greedy generation
through the entry point and its scheduler.
"""
import copy
import json
import os
import random

import numpy as np
import pytest
import torch

import helpers
import plain_zoporax as P

pytestmark = pytest.mark.gpu


def moe(experts, top, ff, scale=1.7, groups=None, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if scale is not None:
        d["router"]["scale"] = scale
    if groups:
        d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def dense(ff):
    return {"kind": "dense", "ff": ff}


YARN = {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}


def latent(heads=3, dim=10, rot_dim=6, vdim=14, kv_rank=20, q_rank=12, dims=None, base=300.0, scale=0.3, scaling=YARN, window=21, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "rot": {"base": base, "dims": rot_dim if dims is None else dims}, "scale": scale}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def linear(heads=3, dim=10, vdim=7, decay=None, mlp=None):
    if decay is None:
        decay = [1.0 - 2.0 ** (-1.0 - 2.0 * i) for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def config_of(layers, width=48, vocab=90, eps=1e-5):
    return {"architecture": "Zoporax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": copy.deepcopy(layers)}


ALONE = {
    "latent": [latent()],
    "latent_part_rot": [latent(heads=2, dim=4, rot_dim=8, vdim=5, kv_rank=9, q_rank=7, dims=4, window=None, scaling=None, mlp=dense(40))],
    "latent_one_key": [latent(heads=1, dim=6, rot_dim=2, vdim=1, kv_rank=5, q_rank=3, window=1, mlp=None)],
    "linear": [linear()],
    "linear_ends": [linear(heads=3, dim=1, vdim=20, decay=[0.0, 1.0, 0.5], mlp=None)],
    "linear_eights": [linear(heads=2, dim=24, vdim=40, decay=[0.9, 0.996], mlp=moe(6, 2, 12, groups=(3, 2), shared=20))],
    "routed": [linear(heads=1, dim=4, vdim=4, decay=[0.8], mlp=moe(5, 3, 9, scale=None)), linear(heads=2, dim=3, vdim=5, decay=[0.7, 0.2], mlp=moe(4, 2, 10, groups=(4, 3)))],
    "dense": [linear(heads=2, dim=4, vdim=4, decay=[0.5, 0.9], mlp=dense(33)), latent(heads=2, mlp=dense(7))],
}
MIXED = [latent(mlp=dense(64)), linear(heads=4, dim=6, vdim=10, mlp=moe(6, 2, 16, groups=(2, 1), shared=24)),
         latent(heads=2, dim=16, rot_dim=4, vdim=8, kv_rank=24, q_rank=20, dims=2, window=50, mlp=moe(9, 1, 20, scale=0.6, groups=(3, 2), shared=20)),
         linear(heads=2, dim=16, vdim=8, decay=[0.3, 0.99], mlp=dense(50)),
         latent(heads=5, dim=3, rot_dim=10, vdim=6, window=16, scaling=None, mlp=None)]
WIDE = [latent(heads=4, dim=48, rot_dim=16, vdim=72, kv_rank=96, q_rank=136, scale=0.12, window=100, mlp=moe(12, 3, 128, groups=(4, 2), shared=384)),
        linear(heads=4, dim=40, vdim=64, mlp=dense(392)),
        linear(heads=2, dim=72, vdim=136, decay=[0.9, 0.995], mlp=moe(6, 2, 136, groups=(2, 1), shared=192)),
        latent(heads=2, dim=64, rot_dim=24, vdim=128, kv_rank=64, q_rank=128, dims=8, scale=0.1, window=None, mlp=None)]
CONFIGS = {
    "mixed": config_of(MIXED),
    "other": config_of([MIXED[3], MIXED[0], MIXED[2], MIXED[1]], width=72, vocab=150, eps=1e-6),
    # wide enough for the tensor-core products of the bfloat16 path
    "wide": config_of(WIDE, width=264, vocab=500),
}


def louder(model_dir, sharp=1.0):
    """The random-weights mode draws small values (standard deviation 0.02) and ones: every softmax would be flat, the
    router near a tie everywhere, every activation linear.  What feeds scores, routers, gates and activations is multiplied up so
    that the mechanisms bite; ``sharp`` multiplies queries and keys further."""
    from cajeta_llm_b200.weights.safetensors_io import Checkpoint, write_safetensors
    ck = Checkpoint(model_dir)
    tensors = {n: ck.load(n).float() for n in ck.names()}
    ck.close()
    for n, t in tensors.items():
        leaf = n.split(".")[-1]
        g = torch.Generator().manual_seed(len(n) + 7 * t.numel())
        if leaf in ("router", "sg"):
            t *= 15.0
        elif leaf == "embed":
            t *= 25.0
        elif leaf in ("uq", "dq"):
            t *= 5.0 * sharp
        elif leaf in ("uk", "dkv"):
            t *= 5.0 * (1.0 if sharp == 1.0 else 3.0)
        elif leaf in ("q", "k", "v", "up", "down", "uv", "o", "gate", "g"):
            t *= 6.0
        elif leaf == "b":
            t.copy_(0.4 * torch.randn(t.shape, generator=g))
        elif leaf in ("norm", "norm1", "norm2"):
            t += 0.3 * torch.randn(t.shape, generator=g)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), {n: t.to(torch.bfloat16) for n, t in tensors.items()})


def sharp(model_dir):
    louder(model_dir, sharp=6.0)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, raw, seed=5, touch=louder):
        if name not in made:
            d = str(tmp_path_factory.mktemp(f"zoporax_{name}"))
            helpers.write_model(d, raw, seed=seed)
            if touch is not None:
                touch(d)
            made[name] = (d, P.load_folder(d))
        return made[name]
    return get


def runner_for(model_dir, dtype, max_seqs=4, max_tokens=512, num_pages=None, cuda_graphs=True, page=16):
    import cajeta_llm_b200  # noqa: F401
    from cajeta_llm_b200.engine.model import load_model
    from cajeta_llm_b200.engine.step import ModelRunner
    from cajeta_llm_b200.parts.base import Runtime
    model, _ = load_model(model_dir, Runtime(dtype, "cuda:0"))
    return ModelRunner(model, page_tokens=page, max_seqs=max_seqs, max_tokens_per_seq=max_tokens,
                       num_pages=num_pages if num_pages is not None else -(-max_tokens // page) * max_seqs, cuda_graphs=cuda_graphs)


def oracle(cfg, W, tokens):
    """The plain implementation's logits and its picks by the engine's routing keys."""
    picks = {}
    want = torch.from_numpy(P.forward(cfg, W, tokens, picks=picks))
    return want, {k: torch.tensor(v, dtype=torch.int32) for k, v in picks.items()}


def pin_rows(spans):
    """A step's routing pin from [(request's picks, first position, count)] in the step's order."""
    if not spans or not spans[0][0]:
        return None
    return {key: torch.cat([p[key][lo:lo + n] for p, lo, n in spans]).cuda().contiguous() for key in spans[0][0]}


def feed(runner, slot, tokens, cuts, picks=None):
    from cajeta_llm_b200.engine.step import StepEntry
    out, at = [], 0
    for n in cuts:
        pin = pin_rows([(picks, at, n)]) if picks else None
        out.append(runner.step([StepEntry(slot, tokens[at:at + n], list(range(n)))], routing_pin=pin).cpu())
        at += n
    assert at == len(tokens)
    return torch.cat(out)


def rel_err(got, want):
    """Per row: RMS of the difference (mean taken off) over the RMS of the wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(dim=-1, keepdim=True)
    w = want.double() - want.double().mean(dim=-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def check(got, want, dtype, what, free_routing=False):
    """float32: every row to rounding.  bfloat16 with the routing pinned: the median row within 5 % of the logits'
    spread, at most a tenth of the rows (or three) beyond 12 %, none beyond 60 % (the weights are loud; a lost key or a
    lost state moves most rows by the logits' whole spread, and the float32 runs hold every row).  With the routing free
    a row near a tie may swap an expert: only the bulk is held."""
    e = rel_err(got, want)
    if dtype == "float32":
        assert float(e.max()) < 1e-4, f"{what}: worst row {int(e.argmax())} differs by {float(e.max()):.2e}"
        return
    over = int((e > 0.12).sum())
    allowed = max(3, int((0.2 if free_routing else 0.1) * e.numel()))
    assert float(e.median()) < 5e-2 and over <= allowed and (free_routing or float(e.max()) < 0.6), \
        f"{what}: median {float(e.median()):.3f}, worst {float(e.max()):.3f} (row {int(e.argmax())}), over 0.12: {over} of {e.numel()}"


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone_as_a_small_model(folders, name):
    d, (cfg, W) = folders(name, config_of(ALONE[name]), seed=3)
    toks = helpers.random_tokens(90, 83, seed=1)
    want, picks = oracle(cfg, W, toks)
    for dtype in ("float32", "bfloat16"):
        pins = picks if dtype == "bfloat16" else None
        r = runner_for(d, dtype, max_tokens=96)
        s = r.admit()
        check(feed(r, s, toks, [83], pins), want, dtype, f"{name} whole {dtype}")
        r.release(s)
        s = r.admit()                                  # the same slot and pages again
        check(feed(r, s, toks, [5, 2, 17, 2, 3, 30] + [1] * 24, pins), want, dtype, f"{name} portions {dtype}")


def test_the_mechanisms_bite(folders):
    """The tests' weights make every mechanism count: an oracle without one of them differs."""
    d, (cfg, W) = folders("mixed", CONFIGS["mixed"], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 90, seed=2)
    want = torch.from_numpy(P.forward(cfg, W, toks))

    def without(change):
        c, w = copy.deepcopy(cfg), dict(W)
        change(c, w)
        return float(rel_err(torch.from_numpy(P.forward(c, w, toks)), want)[30:].max())

    mixer = lambda c, i: c["layers"][i]["mixer"]
    router = lambda c, i: c["layers"][i]["mlp"]["router"]
    for i, window in ((0, 20), (0, 22), (2, 49), (2, 51), (4, 15), (4, 17)):
        assert without(lambda c, w: mixer(c, i)["mask"].update(size=window)) > 1e-3, (i, window)
    assert without(lambda c, w: mixer(c, 4).pop("mask")) > 1e-3
    assert without(lambda c, w: mixer(c, 2)["rot"].update(dims=4)) > 1e-3
    assert without(lambda c, w: mixer(c, 0)["rot"].update(base=1e6)) > 1e-3
    assert without(lambda c, w: mixer(c, 0)["rot"].pop("scaling")) > 1e-3
    assert without(lambda c, w: mixer(c, 0)["rot"]["scaling"].update(factor=4.0)) > 1e-3
    assert without(lambda c, w: mixer(c, 0)["rot"]["scaling"].update(original=512)) > 1e-3
    assert without(lambda c, w: w.update({"l0.mix.g": 0.0 * w["l0.mix.g"]})) > 1e-3
    assert without(lambda c, w: w.update({"l0.mix.dq.norm": np.ones_like(w["l0.mix.dq.norm"])})) > 1e-3
    assert without(lambda c, w: mixer(c, 1)["decay"].__setitem__(3, 0.9)) > 1e-3
    assert without(lambda c, w: w.update({"l1.mix.norm": np.ones_like(w["l1.mix.norm"])})) > 1e-3
    assert without(lambda c, w: w.update({"l1.mix.g": 0.0 * w["l1.mix.g"]})) > 1e-3
    assert without(lambda c, w: router(c, 1).update(scale=1.0)) > 1e-3
    assert without(lambda c, w: router(c, 1).pop("groups")) > 1e-3
    assert without(lambda c, w: c["layers"][1]["mlp"].pop("shared")) > 1e-3
    assert without(lambda c, w: w.update({"l1.mlp.shared.sg": 0.0 * w["l1.mlp.shared.sg"]})) > 1e-3
    for b in ("gate.b", "up.b", "down.b"):
        assert without(lambda c, w: w.update({"l0.mlp." + b: 0.0 * w["l0.mlp." + b]})) > 1e-3, b


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_decoded_and_in_portions(folders, name, dtype):
    d, (cfg, W) = folders(name, CONFIGS[name], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 150, seed=2)
    want, picks = oracle(cfg, W, toks)
    r = runner_for(d, dtype, max_tokens=160)
    results = []
    for cuts in ([150], [86] + [1] * 64, [2] * 75, [7, 2, 16, 3, 2, 9, 5, 2, 15, 14, 33, 2, 40]):
        s = r.admit()
        results.append(feed(r, s, toks, cuts))                       # routing free: steps replay from graphs in bfloat16
        check(results[-1], want, dtype, f"{name} {dtype} cuts {cuts[:4]}", free_routing=True)
        r.release(s)
        if dtype == "bfloat16":
            s = r.admit()
            check(feed(r, s, toks, cuts, picks), want, dtype, f"{name} {dtype} cuts {cuts[:4]}, routing pinned")
            r.release(s)
    if dtype == "float32":
        for other in results[1:]:                                    # the cut changes nothing but the rounding of sums
            assert float(rel_err(other, results[0]).max()) < 2e-5


def test_unequal_requests_in_one_batch_slots_and_pages_used_again(folders):
    """Up to four live requests, portions of some beside single tokens of others, requests that sit a step
    out, in a pool so small that pages and slots come back into use: every position equals the plain
    implementation's."""
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("mixed", CONFIGS["mixed"], seed=7)
    rng = random.Random(4)
    lens = [23, 48, 17, 64, 35, 29, 52, 2, 41, 1]
    toks = {i: helpers.random_tokens(cfg["vocab"], n, seed=50 + i) for i, n in enumerate(lens)}
    both = {i: oracle(cfg, W, t) for i, t in toks.items()}
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_seqs=4, max_tokens=64, num_pages=14)
        waiting, live, got = list(toks), {}, {i: [] for i in toks}
        while waiting or live:
            while waiting and len(live) < 4:
                i = waiting[0]
                if sum(-(-(len(toks[j]) + 15) // 16) for j in live) + -(-(len(toks[i]) + 15) // 16) > 14:
                    break
                waiting.pop(0)
                live[i] = [r.admit(), 0, max(1, len(toks[i]) - rng.randint(3, 12))]
            entries, who, spans = [], [], []
            for i, st in list(live.items()):
                if len(live) > 1 and rng.random() < 0.2:
                    continue
                n = 1 if st[1] >= st[2] else min(rng.randint(2, 11), st[2] - st[1])
                entries.append(StepEntry(st[0], toks[i][st[1]:st[1] + n], list(range(n))))
                who.append((i, n))
                spans.append((both[i][1], st[1], n))
                st[1] += n
            if not entries:
                continue
            out = r.step(entries, routing_pin=pin_rows(spans) if dtype == "bfloat16" else None).cpu()
            at = 0
            for i, n in who:
                got[i].append(out[at:at + n])
                at += n
                if live[i][1] == len(toks[i]):
                    r.release(live.pop(i)[0])
        for i in toks:
            check(torch.cat(got[i]), both[i][0], dtype, f"request {i} in the mixed batch ({dtype})")
        r.cache.books.check()


FAR = {
    "window": [latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=16, q_rank=8, base=10000.0, scale=0.6, window=48, scaling=None)],
    "odd_window": [latent(heads=3, dim=16, rot_dim=4, vdim=24, kv_rank=24, q_rank=16, base=10000.0, scale=0.5, window=67)],
    "no_window": [latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=16, q_rank=8, base=10000.0, scale=0.6, window=None)],
}


@pytest.mark.parametrize("name", sorted(FAR))
def test_window_edges_page_borders_and_far_keys(folders, name):
    """Scores made sharp: a row's output is then close to the value of its best key, which for many rows is about to leave
    the window, lies in another page or chunk of keys, or far back.  Every row equals the plain implementation's, whole, cut
    anywhere - at page borders and one token beside them - and decoded one by one; an oracle whose window is one token
    off, or which forgets the oldest keys, is told apart by a wide margin."""
    # a vocabulary large enough that a token seldom comes twice: keys are then one of a kind
    d, (cfg, W) = folders("far_" + name, config_of(FAR[name], width=32, vocab=2000), seed=9, touch=sharp)
    toks = helpers.random_tokens(2000, 307, seed=5)
    want = torch.from_numpy(P.forward(cfg, W, toks))
    window = cfg["layers"][0]["mixer"].get("mask", {}).get("size")
    if window:
        for other in (window - 1, window + 1):
            c = copy.deepcopy(cfg)
            c["layers"][0]["mixer"]["mask"]["size"] = other
            e = rel_err(torch.from_numpy(P.forward(c, W, toks)), want)
            assert float(e.max()) > 0.1 and int((e > 0.05).sum()) >= 3, "the test's weights do not show the window's edge"
            assert float(e[:window - 1].max()) < 1e-9
    else:
        short = torch.from_numpy(P.forward(cfg, W, toks[40:]))
        assert float(rel_err(short[160:], want[200:]).max()) > 0.1, "the test's weights do not show the far keys"
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=320)
        for cuts in ([307], [300, 4] + [1] * 3, [17] * 18 + [1], [16, 1, 15, 32, 31, 2, 63, 64, 65] + [1] * 18, [30] + [1] * 277):
            s = r.admit()
            check(feed(r, s, toks, cuts), want, dtype, f"far keys {dtype} cuts {cuts[:3]}")
            r.release(s)


def test_a_windowed_request_gives_pages_back(folders):
    """A pool that holds a window and little more: a request much longer than the pool runs through it."""
    d, (cfg, W) = folders("far_window", config_of(FAR["window"], width=32, vocab=2000), seed=9, touch=sharp)
    toks = helpers.random_tokens(2000, 307, seed=5)
    want = torch.from_numpy(P.forward(cfg, W, toks))
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=320, max_seqs=2, num_pages=6)
        s = r.admit()
        check(feed(r, s, toks, [30, 2, 17, 9, 31, 16, 32] + [1] * 170), want, dtype, f"a pool of 96 tokens ({dtype})")
        r.release(s)
        r.cache.books.check()


def test_a_memory_that_reaches_far_back(folders):
    """Decays close to one: what a token left in the state still shows hundreds of tokens later, whole, in portions and
    decoded; an oracle that starts later is told apart."""
    layers = [linear(heads=2, dim=16, vdim=24, decay=[0.9999, 0.99]), linear(heads=3, dim=8, vdim=8, decay=[1.0, 0.999, 0.0])]
    d, (cfg, W) = folders("memory", config_of(layers, width=32, vocab=300), seed=9)
    toks = helpers.random_tokens(300, 700, seed=5)
    want = torch.from_numpy(P.forward(cfg, W, toks))
    short = torch.from_numpy(P.forward(cfg, W, toks[100:]))
    assert float(rel_err(short[400:], want[500:]).max()) > 0.03
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=704, max_seqs=2)
        for cuts in ([700], [300, 200, 64, 65, 33, 32] + [1] * 6, [2] * 30 + [640]):
            s = r.admit()
            check(feed(r, s, toks, cuts), want, dtype, f"memory {dtype} cuts {cuts[:3]}")
            r.release(s)


def test_first_tokens_and_long_decoding(folders):
    d, (cfg, W) = folders("other", CONFIGS["other"], seed=7)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=192)
        for n, cuts in [(n, c) for n in (1, 2, 3, 4, 6) for c in ([1] * n, [n])] + [(183, [3] + [1] * 180)]:
            toks = helpers.random_tokens(cfg["vocab"], n, seed=20 + n)
            want, picks = oracle(cfg, W, toks)
            s = r.admit()
            check(feed(r, s, toks, cuts, picks if dtype == "bfloat16" else None), want, dtype, f"{n} tokens, cuts {cuts[:3]} ({dtype})")
            r.release(s)


def test_captured_steps_equal_uncaptured_ones(folders):
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("wide", CONFIGS["wide"], seed=7)
    toks = [helpers.random_tokens(cfg["vocab"], 100, seed=70 + i) for i in range(3)]
    outs = []
    for graphs in (True, False):
        r = runner_for(d, "bfloat16", max_tokens=128, cuda_graphs=graphs)
        slots = [r.admit() for _ in toks]
        got = []
        for lo, hi in ((0, 12), (12, 24), (24, 36), (36, 48)):       # the same shape again and again: captured, then replayed
            got.append(r.step([StepEntry(s, t[lo:hi], [hi - lo - 1]) for s, t in zip(slots, toks)]).cpu())
        for i in range(48, 100):
            got.append(r.step([StepEntry(s, [t[i]], [0]) for s, t in zip(slots, toks)]).cpu())
        outs.append(torch.cat(got))
        if graphs:
            assert r.graph_replays > 0
    assert torch.equal(outs[0], outs[1])


def test_long_prompts_on_the_tensor_core_attention(folders):
    """Steps of some hundred rows on the bfloat16 path take the tiled attention kernels: a prompt of 700 tokens whole, in
    portions of 300 and 256 beside a second request, and decoded on, against the plain implementation."""
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("wide", CONFIGS["wide"], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 700, seed=12)
    other = helpers.random_tokens(cfg["vocab"], 40, seed=13)
    want, picks = oracle(cfg, W, toks)
    want_other, picks_other = oracle(cfg, W, other)
    for dtype in ("bfloat16", "float32"):
        pins = picks if dtype == "bfloat16" else None
        r = runner_for(d, dtype, max_tokens=768, max_seqs=2)
        s = r.admit()
        check(feed(r, s, toks, [700], pins), want, dtype, f"700 tokens whole ({dtype})")
        r.release(s)
        s, s2 = r.admit(), r.admit()
        got, got2, at = [], [], 0
        for n, m in ((300, 17), (256, 1), (130, 22), (14, 0)):
            entries = [StepEntry(s, toks[at:at + n], list(range(n)))]
            spans = [(picks, at, n)]
            lo = sum(g.shape[0] for g in got2)
            if m:
                entries.append(StepEntry(s2, other[lo:lo + m], list(range(m))))
                spans.append((picks_other, lo, m))
            out = r.step(entries, routing_pin=pin_rows(spans) if dtype == "bfloat16" else None).cpu()
            got.append(out[:n])
            if m:
                got2.append(out[n:])
            at += n
        check(torch.cat(got), want, dtype, f"700 tokens in portions beside another request ({dtype})")
        check(torch.cat(got2), want_other, dtype, f"the other request ({dtype})")


def test_greedy_generation_through_the_entry_point_and_its_scheduler(folders):
    from cajeta_llm_b200.engine.llm_engine import LlmEngine
    from cajeta_llm_b200.engine.options import EngineOptions
    from cajeta_llm_b200.sampling.params import SamplingParams
    d, (cfg, W) = folders("mixed", CONFIGS["mixed"], seed=7)
    prompts = [helpers.random_tokens(cfg["vocab"], n, seed=90 + n) for n in (5, 9, 17, 30, 3, 12)]
    want = [P.greedy(cfg, W, p, 6) for p in prompts]
    # more requests than slots, portions of at most 8 tokens under a budget of 24 a step
    eng = LlmEngine.load(EngineOptions(model=d, dtype="float32", ctx=64, max_seqs=3, chunk=8, max_batch_tokens=24))
    got = eng.generate(prompts, SamplingParams(max_new_tokens=6, stop_token_ids=()))
    assert got == want
    eng.close()
    eng = LlmEngine.load(EngineOptions(model=d, dtype="bfloat16", ctx=64, max_seqs=4))
    got = eng.generate(prompts, SamplingParams(max_new_tokens=6, stop_token_ids=()))
    same = sum(g == w for g, w in zip(got, want))
    assert same >= len(prompts) - 2, f"bfloat16 greedy tokens differ for {len(prompts) - same} prompts"
    eng.close()


def test_replay_tool_on_a_model_folder(folders, tmp_path):
    d, (cfg, W) = folders("other", CONFIGS["other"], seed=7)
    a, b = helpers.random_tokens(cfg["vocab"], 20, seed=1), helpers.random_tokens(cfg["vocab"], 9, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:11], "want": [10]}, {"id": "b", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[11:], "want": [0, 8]}], "end": ["a"]}]
    import subprocess
    import sys
    cmd = [sys.executable, os.path.join(helpers.ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(tmp_path),
           "--max-tokens", "128"]
    proc = subprocess.run(cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = oracle(cfg, W, a)[0], oracle(cfg, W, b)[0]
    got = {n: torch.from_numpy(np.fromfile(os.path.join(str(tmp_path), f"{n}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])) for n in range(3)}
    check(got[0], wa[10:11], "float32", "step 0")
    check(got[1], wb[8:9], "float32", "step 1")
    check(got[2], wa[[11, 19]], "float32", "step 2")


def random_config(seed):
    """A configuration drawn at random: layer order, every size and constant."""
    rng = random.Random(seed)
    width = rng.choice([40, 72, 136, 256])
    big = width >= 128

    def pick(lo, hi):
        return rng.randint(lo, hi)

    layers = []
    for i in range(rng.randint(1, 5)):
        mlp = None
        u = rng.random()
        if u < 0.5:
            per, count = pick(1, 4), pick(1, 5)
            keep = pick(1, count)
            mlp = moe(per * count, pick(1, per * keep), rng.choice([pick(8, 60), 128, 136]) if big else pick(8, 60), scale=rng.choice([None, 0.5, 2.5]),
                      groups=rng.choice([None, (count, keep)]) if count > 1 else None, shared=rng.choice([None, pick(8, 60), 128 if big else 24]))
        elif u < 0.8:
            mlp = dense(rng.choice([pick(8, 80), 256]) if big else pick(8, 80))
        if rng.random() < 0.45:
            heads = pick(1, 5)
            layers.append(linear(heads=heads, dim=rng.choice([16, 32, 64, 96]) if big and rng.random() < 0.6 else pick(1, 24),
                                 vdim=rng.choice([32, 64, 80, 144]) if big and rng.random() < 0.6 else pick(1, 40),
                                 decay=[rng.choice([0.0, 0.3, 0.9, 0.99, 0.999, 1.0]) for _ in range(heads)], mlp=mlp))
        else:
            rot_dim = 2 * pick(1, 16)
            layers.append(latent(heads=pick(1, 5), dim=rng.choice([32, 64]) if big and rng.random() < 0.5 else pick(2, 24), rot_dim=rot_dim,
                                 vdim=rng.choice([32, 64, 96]) if big and rng.random() < 0.5 else pick(2, 24),
                                 kv_rank=rng.choice([64, 128]) if big and rng.random() < 0.5 else pick(4, 48), q_rank=pick(2, 40),
                                 dims=rot_dim if rng.random() < 0.6 else 2 * pick(1, rot_dim // 2), base=rng.choice([100.0, 10000.0, 500000.0]),
                                 scaling=rng.choice([None, {"factor": rng.choice([2.0, 8.0]), "original": rng.choice([32, 512]), "fast": 16.0, "slow": 1.0}]),
                                 scale=rng.choice([0.1, 0.3]), window=rng.choice([None, pick(1, 70)]), mlp=mlp))
    return config_of(layers, width=width, vocab=rng.choice([70, 131, 300]), eps=rng.choice([1e-5, 1e-6]))


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(folders, seed):
    raw = random_config(7000 + seed)
    d, (cfg, W) = folders(f"random{seed}", raw, seed=100 + seed)
    toks = helpers.random_tokens(cfg["vocab"], 120, seed=seed)
    want, picks = oracle(cfg, W, toks)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=128)
        for cuts in ([120], [17, 2, 9, 60] + [1] * 32):
            s = r.admit()
            check(feed(r, s, toks, cuts, picks if dtype == "bfloat16" else None), want, dtype,
                  f"{json.dumps(raw)} {dtype} cuts {cuts[:3]}")
            r.release(s)


def _cuda(*ts):
    return [t.cuda() for t in ts]


@pytest.mark.parametrize("heads,dim,vdim,requests", [
    (3, 10, 7, [5, 0, 1, 40]),
    (2, 64, 64, [300, 1, 33, 32]),
    (4, 128, 128, [700, 64, 65]),
    (2, 40, 72, [129, 5, 200]),
    (1, 128, 200, [1000]),
    (5, 8, 8, [1] * 9),
    (2, 200, 16, [70, 3]),
])
def test_decay_attention_against_the_recurrence(heads, dim, vdim, requests):
    """The walk in both dtypes, and the chunks on the tensor cores with segments of several lengths, from a state that is not
    zero, with a slot that is not the request's number and an absent request, against the recurrence token by token."""
    from cajeta_llm_b200.csrc import kernels as K
    rng = np.random.default_rng(heads * 1000 + dim + vdim)
    T, slots = sum(requests), len(requests) + 2
    dec = rng.choice([0.0, 0.4, 0.93, 0.999, 1.0], size=heads)
    ld = heads * (2 * dim + vdim) + 16
    x = torch.from_numpy(rng.normal(size=(T, ld)) * 0.7).to(torch.bfloat16)
    off = (8, 8 + heads * dim, 8 + 2 * heads * dim)
    state0 = torch.from_numpy(rng.normal(size=(slots, 24 + heads * dim * vdim))).float()
    slot_of = rng.permutation(slots)[:len(requests)].tolist()
    q, k, v = (x.double().numpy()[:, o:o + heads * n].reshape(T, heads, n) for o, n in zip(off, (dim, dim, vdim)))
    want, after, at = np.zeros((T, heads, vdim)), state0.double().numpy().copy(), 0
    for r, n in enumerate(requests):
        S = after[slot_of[r], 24:].reshape(heads, dim, vdim)
        for t in range(at, at + n):
            S[:] = dec[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            want[t] = np.einsum("hdv,hd->hv", S, q[t])
        at += n
    starts = torch.tensor(np.concatenate([[0], np.cumsum(requests), [T]]), dtype=torch.int32).cuda()      # one more request, absent
    slot_t = torch.tensor(slot_of + [-1], dtype=torch.int32).cuda()
    tables = [torch.from_numpy(t).cuda() for t in (dec.astype(np.float32), (dec[:, None] ** np.arange(65)[None]).astype(np.float32))]
    with np.errstate(divide="ignore"):
        l2 = torch.from_numpy(np.log2(dec)).cuda()
    scale = float(np.sqrt((want ** 2).mean()))
    runs = [(torch.float32, False, 0), (torch.bfloat16, False, 0)]
    if K.decay_chunk_shape(dim, vdim) and ld % 8 == 0:
        runs += [(torch.bfloat16, True, seg) for seg in (0, 64, 192, 4096)]
    for dtype, chunked, seg in runs:
        st, out = state0.clone().cuda(), torch.full((T, heads * vdim), float("nan"), device="cuda")
        K.decay_attention(x.to(dtype).cuda(), *off, tables[0], tables[1], l2, st, 24, starts, slot_t, len(requests) + 1, out, heads, dim, vdim,
                          segment=seg, chunked=chunked)
        tol = 1e-4          # float32 sums over up to a thousand tokens, some of which never fade; chunks: two bfloat16 terms a value
        err = np.abs(out.cpu().double().numpy().reshape(want.shape) - want).max() / scale
        assert err < tol, f"{dtype} chunked={chunked} segments of {seg}: outputs differ by {err:.2e}"
        err = np.abs(st.cpu().double().numpy() - after).max() / np.abs(after).max()
        assert err < tol, f"{dtype} chunked={chunked} segments of {seg}: states differ by {err:.2e}"


def test_row_norm_with_a_gate():
    from cajeta_llm_b200.csrc import kernels as K
    for n, dtype in ((7, torch.float32), (300, torch.bfloat16), (4096, torch.bfloat16)):
        g = torch.Generator().manual_seed(n)
        y, z, w = torch.randn((5, n), generator=g), torch.randn((5, n + 9), generator=g).to(dtype), torch.randn(n, generator=g)
        out = torch.empty((5, n), dtype=dtype, device="cuda")
        K.gated_row_norm(*_cuda(y, z), 9, w.cuda(), 1e-5, out)
        yd = y.double()
        want = yd / torch.sqrt((yd * yd).mean(-1, keepdim=True) + 1e-5) * w.double() * torch.sigmoid(z[:, 9:].double())
        assert float((out.cpu().double() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())


@pytest.mark.parametrize("rows", [1, 5, 40, 700])
@pytest.mark.parametrize("features,inner", [(136, 136), (264, 392), (30, 24)])
def test_gated_products_with_gelu_and_biases(rows, features, inner):
    """gelu_tanh(x Wg + bg) * (x Wu + bu) on every product kernel: both dtypes, few and many rows, and pairs of SMs."""
    from cajeta_llm_b200.csrc import kernels as K
    from cajeta_llm_b200.parts.base import Runtime
    from cajeta_llm_b200.parts.linear import project
    g = torch.Generator().manual_seed(rows + features)
    x, wg, wu = (torch.randn(s, generator=g).bfloat16() for s in ((rows, inner), (features, inner), (features, inner)))
    wg, wu = wg * 0.15, wu * 0.15
    bg, bu = torch.randn(features, generator=g), torch.randn(features, generator=g)
    a, u = x.double() @ wg.double().T + bg.double(), x.double() @ wu.double().T + bu.double()
    want = 0.5 * a * (1.0 + torch.tanh((2.0 / np.pi) ** 0.5 * (a + 0.044715 * a ** 3))) * u
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 1.2e-2)):
        rt = Runtime(dtype, "cuda:0")
        out = torch.empty((rows, features), dtype=rt.act_dtype, device="cuda")
        project(rt, x.to(rt.act_dtype).cuda(), rt.matrix(wg), out, w_up=rt.matrix(wu), bias=bg.cuda(), bias_up=bu.cuda(),
                act_alpha=K.GELU_TANH[0], act_cubic=K.GELU_TANH[1])
        err = (out.cpu().double() - want).abs().max() / want.abs().max()
        assert float(err) < tol, f"{dtype}: {float(err):.2e}"


@pytest.mark.parametrize("rows", [1, 17, 130, 900])
@pytest.mark.parametrize("act,features,inner,first", [("gelu", 256, 136, 0), ("silu", 520, 264, 300), ("relu2", 264, 128, 0), ("gelu", 20, 24, 0), ("silu", 33, 30, 17)])
def test_activations_of_a_product(rows, act, features, inner, first):
    from cajeta_llm_b200.parts.base import Runtime
    from cajeta_llm_b200.parts.linear import project
    g = torch.Generator().manual_seed(rows + features)
    x, w, b = torch.randn((rows, inner), generator=g).bfloat16(), (torch.randn((features, inner), generator=g) * 0.15).bfloat16(), torch.randn(features, generator=g)
    z = x.double() @ w.double().T + b.double()
    f = {"gelu": lambda v: 0.5 * v * (1.0 + torch.erf(v / 2.0 ** 0.5)), "silu": lambda v: v * torch.sigmoid(v), "relu2": lambda v: v.clamp_min(0.0) ** 2}[act]
    want = f(z)
    if first:
        want[:, first:] = z[:, first:]
    for dtype, tol in (("float32", 1e-5), ("bfloat16", 6e-3)):
        rt = Runtime(dtype, "cuda:0")
        out = torch.empty((rows, features), dtype=rt.act_dtype, device="cuda")
        project(rt, x.to(rt.act_dtype).cuda(), rt.matrix(w), out, bias=b.cuda(), act=act, act_features=first)
        err = (out.cpu().double() - want).abs() / (want.abs() + 0.02 * float(want.abs().max()))
        assert float(err.max()) < tol, f"{dtype}: {float(err.max()):.2e}"


@pytest.mark.parametrize("experts,top,groups", [(12, 3, (4, 2)), (6, 2, (6, 3)), (20, 5, (2, 1)), (40, 4, (5, 3)), (7, 2, None)])
def test_router_with_groups_scored_by_their_two_best(experts, top, groups):
    """Both router kernels (few and many rows) and the selection from partial sums against the plain router; an oracle that
    scores a group by its best alone picks otherwise for some rows."""
    from cajeta_llm_b200.csrc import kernels as K
    rng = np.random.default_rng(experts)
    w = rng.normal(size=(experts, 24)) * 0.3          # scores away from 0 and 1, where float32 would tie
    ff = {"router": {"experts": experts, "top": top, "scale": 1.3}}
    if groups:
        ff["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    for rows in (9, 200):
        x = rng.normal(size=(rows, 24)).astype(np.float32)
        w32 = w.astype(np.float32)
        picks, weights = P.route(x.astype(np.float64), {".router": w32.astype(np.float64)}, "", ff)
        logits = torch.from_numpy(x.astype(np.float64) @ w32.T.astype(np.float64)).float()
        for form in ("rows", "partials"):
            sel, wts = torch.empty((rows, top), dtype=torch.int32, device="cuda"), torch.empty((rows, top), device="cuda")
            kw = dict(sigmoid_scores=True, groups=groups, weight_scale=1.3, group_top2=True, norm_floor=1e-20)
            if form == "rows":
                K.router_topk(torch.from_numpy(x).cuda(), torch.from_numpy(w32).cuda(), None, top, True, sel, wts, None, **kw)
            else:
                parts = torch.stack([logits * 0.25, logits * 0.75]).cuda().contiguous()
                K.router_select(parts, experts, top, True, sel, wts, None, **kw)
            assert sel.cpu().tolist() == picks
            assert np.allclose(wts.cpu().numpy(), weights, rtol=2e-5)
        if groups and experts // groups[0] > 1 and rows == 200:
            sel = torch.empty((rows, top), dtype=torch.int32, device="cuda")
            K.router_topk(torch.from_numpy(x).cuda(), torch.from_numpy(w32).cuda(), None, top, True, sel, torch.empty((rows, top), device="cuda"), None,
                          sigmoid_scores=True, groups=groups)
            assert sel.cpu().tolist() != picks


def _latent_formula(q_abs, q_rot, entries, positions, row_req, rank, window, scale):
    """softmax(q . entry) over the visible entries, times their latents; q_abs [H, T, rank], q_rot [T, H, rot]."""
    H, T, _ = q_abs.shape
    out = torch.zeros((H, T, rank), dtype=torch.float64)
    for t in range(T):
        p, e = int(positions[t]), entries[int(row_req[t])].double()
        lo = max(0, p + 1 - window) if window > 0 else 0
        for h in range(H):
            s = (e[lo:p + 1, :rank] @ q_abs[h, t].double() + e[lo:p + 1, rank:] @ q_rot[t, h].double()) * scale
            out[h, t] = torch.softmax(s, 0) @ e[lo:p + 1, :rank]
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,rank,rot,window,requests", [
    (3, 20, 6, 21, [(0, 40), (20, 1), (21, 1), (22, 1), (100, 3)]),
    (9, 64, 16, 100, [(99, 1), (100, 1), (101, 1), (250, 1), (0, 1)]),
    (2, 33, 4, 1, [(0, 3), (40, 1)]),
    (4, 128, 32, 64, [(63, 1), (64, 1), (65, 1), (500, 2)]),
])
def test_windowed_latent_attention_against_the_formula(dtype, heads, rank, rot, window, requests):
    """The absorbed form on pages in a shuffled order whose pages behind the window are gone (their table entries -1), rows
    just before, on and after the position where the window begins to move, keys cut into stretches or not."""
    from cajeta_llm_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(rank + window)
    page, dev, dt = 16, "cuda", getattr(torch, dtype)
    totals = [p + r for p, r in requests]
    entries = [(torch.randn((t, rank + rot), generator=g) * 0.6).to(dt) for t in totals]
    n_pages = sum(-(-t // page) for t in totals) + 2
    order, table, at = torch.randperm(n_pages, generator=g).tolist(), torch.full((len(requests), -(-max(totals) // page)), -1, dtype=torch.int32), 0
    plane = torch.zeros((n_pages, 1, page, rank + rot), dtype=dt)
    for i, t in enumerate(totals):
        oldest = max(0, requests[i][0] + 1 - window)
        for b in range(-(-t // page)):
            pg, at = order[at], at + 1
            if (b + 1) * page > oldest:
                table[i, b] = pg
            chunk = entries[i][b * page:(b + 1) * page]
            plane[pg, 0, :chunk.shape[0]] = chunk
    positions = torch.cat([torch.arange(p, p + r) for p, r in requests]).int()
    row_req = torch.cat([torch.full((r,), i) for i, (_, r) in enumerate(requests)]).int()
    T = positions.numel()
    q_abs, q_rot = torch.randn((heads, T, rank), generator=g), torch.randn((T, heads, rot), generator=g)
    want = _latent_formula(q_abs, q_rot, entries, positions, row_req, rank, window, 0.7)
    for reach in (0, max(totals)):
        out = torch.full((heads * T, rank), float("nan"), dtype=dt, device=dev)
        K.latent_attention(q_abs.reshape(heads * T, rank).contiguous().to(dev), q_rot.to(dev), plane.to(dev), rank, rot, heads, positions.to(dev),
                           row_req.to(dev), table.to(dev), page, 0.7, out, max_context=reach, window=window)
        err = (out.cpu().double().view(heads, T, rank) - want).abs().max()
        assert float(err) < (2e-5 if dtype == "float32" else 1e-2) * max(1.0, float(want.abs().max())), f"reach {reach}: {float(err):.2e}"
    for other in (window - 1, window + 1):
        if other > 0:
            assert float((_latent_formula(q_abs, q_rot, entries, positions, row_req, rank, other, 0.7) - want).abs().max()) > 0.05


@pytest.mark.parametrize("DK,DV,window,requests", [
    (64, 64, 40, [(0, 130), (39, 5), (300, 70)]),
    (128, 64, 64, [(0, 64), (63, 66), (64, 1), (1000, 3)]),
    (192, 128, 200, [(0, 420), (7, 2)]),
    (64, 128, 1, [(0, 70), (200, 65)]),
    (256, 128, 0, [(0, 100), (77, 60)]),
])
def test_windowed_tiled_latent_attention_against_the_formula(DK, DV, window, requests):
    """The plain form's kernel over dense keys and values that begin with the oldest token a request's rows see, weights in one
    and in two bfloat16 terms (the second within a quarter of the first's error)."""
    from cajeta_llm_b200.csrc import kernels as K
    g, H, dev = torch.Generator().manual_seed(DK + window), 2, "cuda"
    firsts = [max(0, p + 1 - window) if window else 0 for p, _ in requests]
    counts = [p + r - f for (p, r), f in zip(requests, firsts)]
    starts = [0]
    for c in counts:
        starts.append(starts[-1] + c)
    base = torch.tensor([s - f for s, f in zip(starts, firsts)], dtype=torch.int32)
    kx, vx = (torch.randn((starts[-1], H, DK), generator=g) * 0.8).bfloat16(), torch.randn((starts[-1], H, DV), generator=g).bfloat16()
    rows = [0]
    for _, r in requests:
        rows.append(rows[-1] + r)
    q = torch.randn((rows[-1], H, DK), generator=g).bfloat16()
    scale, want = DK ** -0.5, torch.zeros((rows[-1], H, DV), dtype=torch.float64)
    for i, (p, r) in enumerate(requests):
        for j in range(r):
            lo = max(0, p + j + 1 - window) if window else 0
            a, b = int(base[i]) + lo, int(base[i]) + p + j + 1
            for h in range(H):
                want[rows[i] + j, h] = torch.softmax((kx[a:b, h].double() @ q[rows[i] + j, h].double()) * scale, 0) @ vx[a:b, h].double()
    errs = []
    for exact in (False, True):
        out = torch.full((rows[-1], H, DV), float("nan"), dtype=torch.bfloat16, device=dev)
        K.latent_flash(*_cuda(q), out, *_cuda(kx, vx), torch.tensor(rows, dtype=torch.int32, device=dev),
                       torch.tensor([p for p, _ in requests], dtype=torch.int32, device=dev), base.to(dev), len(requests), H, scale, window=window,
                       exact_weights=exact)
        got = out.cpu().double()
        assert float((got - want).abs().max()) < 2e-2 * max(1.0, float(want.abs().max()))
        errs.append(float((got - want).pow(2).mean().sqrt()))
    assert errs[1] <= errs[0] * 1.001


def test_the_fast_gelu_holds_its_bound():
    """The bfloat16 products' gelu before rounding is what the published approximation promises: every bfloat16 input through an
    identity product equals the rounded exact value, or the neighbour where the exact value lies within the bound of a tie."""
    from cajeta_llm_b200.parts.base import Runtime
    from cajeta_llm_b200.parts.linear import project
    rt = Runtime("bfloat16", "cuda:0")
    bits = torch.arange(0, 1 << 16, dtype=torch.int32).to(torch.int16).view(torch.bfloat16)
    vals = bits[torch.isfinite(bits.float()) & (bits.float().abs() < 30.0)]
    n = vals.numel() // 128 * 128
    x = vals[:n].view(-1, 128).contiguous()
    out = torch.empty(x.shape, dtype=torch.bfloat16, device="cuda")
    project(rt, x.cuda(), torch.eye(128, dtype=torch.bfloat16, device="cuda"), out, act="gelu")
    xd = x.double()
    exact = 0.5 * xd * torch.special.erfc(-xd / 2.0 ** 0.5)
    err = (out.cpu().double() - exact).abs()
    assert bool((err <= exact.abs() * 2.0 ** -8 + xd.abs() * 2e-7 + 1e-38).all())
