"""Rugezen through the engine against the plain implementation (``plain_rugezen.py``), and its kernels against formulas.

Small configurations of their own whose sizes differ in every field (head groups, values of another size than keys, a
rotation over a part of the heads, recurrences narrower and wider than the model, layers without a feed-forward, a looped
stretch run two and three times, sizes that are 1 or odd).  Each mechanism alone as a small model; whole prompts against
token-by-token decoding and portions down to two tokens; unequal requests in one batch against each alone; slots and pages
used again; attention made sharp so that single keys - far ones, those at page borders, the first ones - decide a row, and a
recurrence made slow so that far tokens stay in the state, in prompts and in decoding; first tokens; long decoding; greedy
generation through the entry point and its scheduler.
"""
import copy
import json
import math
import os
import random

import numpy as np
import pytest
import torch

import helpers
import plain_rugezen as P

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def attn(heads=4, kv_heads=2, dim=12, vdim=10, dims=6, base=500.0, scale=0.4, softcap=20.0, ff=40):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims}, "scale": scale, "softcap": softcap}
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def gru(width=28, ff=36):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config_of(layers, width=48, vocab=90, eps=1e-5, mult=0.6, loop=None):
    c = {"architecture": "Rugezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": copy.deepcopy(layers)}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


ALONE = {
    "attention": config_of([attn(ff=None)]),
    "attention_all_rotated": config_of([attn(heads=3, kv_heads=3, dim=8, vdim=8, dims=8, base=30.0, ff=24)], mult=1.0),
    "attention_odd": config_of([attn(heads=5, kv_heads=1, dim=7, vdim=9, dims=2, softcap=3.0, scale=0.9, ff=None)], width=30),
    "attention_one": config_of([attn(heads=2, kv_heads=1, dim=2, vdim=1, dims=2, scale=2.0, ff=5)], width=20),
    "mingru": config_of([gru(ff=None)]),
    "mingru_wide": config_of([gru(width=131, ff=50)], width=33, mult=0.3),
    "mingru_one": config_of([gru(width=1, ff=3)], width=16),
    "looped": config_of([gru(20), attn(), gru(33, ff=None)], loop=(0, 2, 3)),
    "looped_one_layer": config_of([attn(), gru(), attn(heads=2, kv_heads=2)], loop=(1, 2, 2)),
    "looped_once": config_of([gru(), attn()], loop=(0, 2, 1)),
}
CONFIGS = {
    "mixed": config_of([attn(), gru(), attn(heads=6, kv_heads=3, dim=16, vdim=24, dims=8, scale=0.25, softcap=8.0, ff=None), gru(width=70, ff=64)],
                       loop=(1, 3, 2)),
    "other": config_of([gru(width=64), attn(heads=3, kv_heads=1, dim=20, vdim=6, dims=20, base=10000.0)], width=72, vocab=150, eps=1e-6, mult=0.22),
    # wide enough for the tensor-core products and tiled attention of the bfloat16 path: head sizes 128, 96 and 40 | 72
    "wide": config_of([attn(heads=4, kv_heads=2, dim=128, vdim=128, dims=64, scale=0.12, softcap=30.0, ff=384), gru(width=200, ff=512),
                       attn(heads=3, kv_heads=1, dim=96, vdim=96, dims=40, scale=0.11, softcap=12.0, ff=256),
                       attn(heads=4, kv_heads=4, dim=40, vdim=72, dims=10, scale=0.2, softcap=9.0, ff=None)], width=256, vocab=500, loop=(0, 2, 2)),
}


def louder(model_dir, sharp=1.0, slow=False):
    """The random-weights mode draws small values (standard deviation 0.02) and ones: every gate would stand at its bias, every
    residual branch be a whisper.  What feeds gates and branches is multiplied up so that the mechanisms bite.  ``slow``: the
    recurrences' gates lie near zero except where a token opens them, so that a far token stays in the state."""
    from cajeta_llm_b200.weights.safetensors_io import Checkpoint, write_safetensors
    ck = Checkpoint(model_dir)
    tensors = {n: ck.load(n).float() for n in ck.names()}
    ck.close()
    for n, t in tensors.items():
        leaf, g = n.split(".")[-1], torch.Generator().manual_seed(sum(map(ord, n)) + 7 * t.numel())
        if leaf == "embed":
            t *= 50.0
        elif leaf in ("q", "k", "v", "x", "g"):
            t *= 6.0
        elif leaf == "z":
            t *= 8.0 if slow else 10.0
        elif leaf in ("o", "up", "down"):
            t *= 5.0
        elif leaf == "b" and n.split(".")[-2] in ("up", "down"):
            t.copy_(0.3 * torch.randn(t.shape, generator=g))
        elif leaf == "b" and slow and n.split(".")[-2] == "z":
            t.copy_(-6.0 + torch.randn(t.shape, generator=g))
        elif leaf in ("norm", "norm1", "norm2"):
            t += 0.3 * torch.randn(t.shape, generator=g)
    write_safetensors(os.path.join(model_dir, "model.safetensors"), {n: t.to(torch.bfloat16) for n, t in tensors.items()})


def slow(model_dir):
    louder(model_dir, slow=True)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name, raw, seed=5, touch=louder):
        if name not in made:
            d = str(tmp_path_factory.mktemp(f"rugezen_{name}"))
            helpers.write_model(d, raw, seed=seed)
            touch(d)
            made[name] = (d, P.load_folder(d))
        return made[name]

    return get


def runner_for(model_dir, dtype, max_seqs=4, max_tokens=512, num_pages=None, cuda_graphs=True, page=16):
    import cajeta_llm_b200  # noqa: F401
    from cajeta_llm_b200.engine.model import load_model
    from cajeta_llm_b200.engine.step import ModelRunner
    from cajeta_llm_b200.parts.base import Runtime
    model, _ = load_model(model_dir, Runtime(dtype, DEV))
    return ModelRunner(model, page_tokens=page, max_seqs=max_seqs, max_tokens_per_seq=max_tokens,
                       num_pages=num_pages if num_pages is not None else -(-max_tokens // page) * max_seqs, cuda_graphs=cuda_graphs)


def feed(runner, slot, tokens, cuts):
    from cajeta_llm_b200.engine.step import StepEntry
    out, at = [], 0
    for n in cuts:
        out.append(runner.step([StepEntry(slot, tokens[at:at + n], list(range(n)))]).cpu())
        at += n
    assert at == len(tokens)
    return torch.cat(out)


def oracle(cfg, W, tokens):
    return torch.from_numpy(P.forward(cfg, W, tokens))


def rel_err(got, want):
    """Per row: RMS of the difference (mean taken off) over the RMS of the wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(dim=-1, keepdim=True)
    w = want.double() - want.double().mean(dim=-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def check(got, want, dtype, what):
    """float32: every row to rounding.  bfloat16: the median row within 3 % of the logits' spread, none beyond 20 % (a lost
    key or a lost state moves most rows by far more, and the float32 runs hold every row)."""
    e = rel_err(got, want)
    if dtype == "float32":
        assert float(e.max()) < 5e-5, f"{what}: worst row {int(e.argmax())} differs by {float(e.max()):.2e}"
    else:
        assert float(e.median()) < 3e-2 and float(e.max()) < 0.2, \
            f"{what}: median {float(e.median()):.3f}, worst {float(e.max()):.3f} (row {int(e.argmax())})"


@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone_as_a_small_model(folders, name):
    d, (cfg, W) = folders(name, ALONE[name], seed=3)
    toks = helpers.random_tokens(90, 83, seed=1)
    want = oracle(cfg, W, toks)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=96)
        s = r.admit()
        check(feed(r, s, toks, [83]), want, dtype, f"{name} whole {dtype}")
        r.release(s)
        s = r.admit()                                  # the same slot and pages again
        check(feed(r, s, toks, [5, 2, 17, 2, 3, 30] + [1] * 24), want, dtype, f"{name} portions {dtype}")


def test_the_mechanisms_bite(folders, monkeypatch):
    """The tests' weights make every mechanism count: an oracle without one of them differs."""
    d, (cfg, W) = folders("mixed", CONFIGS["mixed"], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 90, seed=2)
    want = oracle(cfg, W, toks)

    def moved(change=None, **patched):
        c, w = copy.deepcopy(cfg), dict(W)
        if change:
            change(c, w)
        with monkeypatch.context() as m:
            for name, fn in patched.items():
                m.setattr(P, name, fn)
            return float(rel_err(oracle(c, w, toks), want)[30:].max())

    mixer = lambda c, i: c["layers"][i]["mixer"]
    plain_softmax = lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum()
    floor = 2e-3                                       # forty times what a float32 row may differ by
    assert moved(softmax_plus_one=plain_softmax) > floor
    assert moved(candidate=lambda u: P.sigmoid(u)) > floor and moved(candidate=lambda u: u + 0.5) > floor
    assert moved(lambda c, w: mixer(c, 0)["rot"].update(base=400.0)) > floor
    assert moved(lambda c, w: mixer(c, 0)["rot"].update(dims=8)) > floor
    assert moved(lambda c, w: mixer(c, 2).update(softcap=80.0)) > floor
    assert moved(lambda c, w: mixer(c, 2).update(scale=0.26)) > floor
    assert moved(lambda c, w: c.update(residual_mult=0.59)) > floor
    assert moved(lambda c, w: c["loop"].update(times=1)) > floor and moved(lambda c, w: c["loop"].update(times=3)) > floor
    assert moved(lambda c, w: c["loop"].update(start=0)) > floor and moved(lambda c, w: c["loop"].update(stop=4)) > floor
    for name in ("l1.mix.z.b", "l1.mix.x.b", "l0.mlp.up.b", "l0.mlp.down.b"):
        assert moved(lambda c, w: w.update({name: 0.0 * w[name]})) > floor, name
    assert moved(lambda c, w: w.update({"l0.norm2": w["l0.norm1"]})) > floor
    unit = P.unit_rms

    def no_value_norm(x, eps):
        return x if x.ndim == 3 and x.shape[-1] == 10 else unit(x, eps)          # layer 0's values have ten entries
    assert moved(unit_rms=no_value_norm) > floor

    def no_head_norm(x, eps):
        return x if x.ndim == 3 and x.shape[-1] == 12 else unit(x, eps)          # and its queries and keys twelve
    assert moved(unit_rms=no_head_norm) > floor


@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_decoded_and_in_portions(folders, name, dtype):
    d, (cfg, W) = folders(name, CONFIGS[name], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 150, seed=2)
    want = oracle(cfg, W, toks)
    r = runner_for(d, dtype, max_tokens=160)
    results = []
    for cuts in ([150], [86] + [1] * 64, [2] * 75, [7, 2, 16, 3, 2, 9, 5, 2, 15, 14, 33, 2, 40]):
        s = r.admit()
        results.append(feed(r, s, toks, cuts))
        check(results[-1], want, dtype, f"{name} {dtype} cuts {cuts[:4]}")
        r.release(s)
    if dtype == "float32":
        for other in results[1:]:                                    # the cut changes nothing but the rounding of sums
            assert float(rel_err(other, results[0]).max()) < 2e-5


@pytest.mark.parametrize("page", [16, 64])
def test_unequal_requests_in_one_batch_slots_and_pages_used_again(folders, page):
    """Up to four live requests, portions of some beside single tokens of others, requests that sit a step out, in a pool so
    small that pages and slots come back into use: every position equals the plain implementation's."""
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("mixed", CONFIGS["mixed"], seed=7)
    rng = random.Random(4)
    lens = [23, 48, 17, 64, 35, 29, 52, 2, 41, 1]
    toks = {i: helpers.random_tokens(cfg["vocab"], n, seed=50 + i) for i, n in enumerate(lens)}
    want = {i: oracle(cfg, W, t) for i, t in toks.items()}
    pool = 14 if page == 16 else 4
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_seqs=4, max_tokens=64, num_pages=pool, page=page)
        waiting, live, got = list(toks), {}, {i: [] for i in toks}
        while waiting or live:
            while waiting and len(live) < 4:
                i = waiting[0]
                if sum(-(-(len(toks[j]) + page - 1) // page) for j in live) + -(-(len(toks[i]) + page - 1) // page) > pool and live:
                    break
                waiting.pop(0)
                live[i] = [r.admit(), 0, max(1, len(toks[i]) - rng.randint(3, 12))]
            entries, who = [], []
            for i, st in list(live.items()):
                if len(live) > 1 and rng.random() < 0.2:
                    continue
                n = 1 if st[1] >= st[2] else min(rng.randint(2, 19), st[2] - st[1])
                entries.append(StepEntry(st[0], toks[i][st[1]:st[1] + n], list(range(n))))
                who.append((i, n))
                st[1] += n
            if not entries:
                continue
            out = r.step(entries).cpu()
            at = 0
            for i, n in who:
                got[i].append(out[at:at + n])
                at += n
                if live[i][1] == len(toks[i]):
                    r.release(live.pop(i)[0])
        for i in toks:
            check(torch.cat(got[i]), want[i], dtype, f"request {i} in the mixed batch ({dtype})")
        r.cache.books.check()


FAR = {
    # scores of up to scale * dim: a row's output is close to the value of its best key
    "attention": config_of([attn(heads=4, kv_heads=2, dim=16, vdim=16, dims=2, base=10000.0, scale=1.5, softcap=60.0, ff=None)], width=32, vocab=2000, mult=1.5),
    "attention_two_sizes": config_of([attn(heads=2, kv_heads=1, dim=24, vdim=40, dims=4, base=10000.0, scale=1.0, softcap=40.0, ff=None)], width=32, vocab=2000, mult=1.5),
    "mingru": config_of([gru(width=40, ff=None)], width=32, vocab=2000, mult=6.0),
    "looped": config_of([attn(heads=2, kv_heads=2, dim=16, vdim=16, dims=2, base=10000.0, scale=1.2, softcap=50.0, ff=None), gru(width=40, ff=None)],
                        width=32, vocab=2000, mult=0.8, loop=(0, 2, 2)),
}


@pytest.mark.parametrize("name", sorted(FAR))
def test_far_tokens_page_borders_and_the_first_tokens(folders, name):
    """A row depends on tokens hundreds of places back, in another page and another tile of keys or of the recurrence, and on
    the very first.  Every row equals the plain implementation's, whole, cut anywhere - at page borders and one token beside
    them - and decoded one by one; an oracle that forgets the oldest tokens is told apart by a wide margin."""
    d, (cfg, W) = folders("far_" + name, FAR[name], seed=9, touch=slow)
    toks = helpers.random_tokens(2000, 307, seed=5)
    want = oracle(cfg, W, toks)
    short = oracle(cfg, W, toks[40:])
    assert float(rel_err(short[160:], want[200:]).max()) > 0.05, "the test's weights do not show the far tokens"
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=320)
        for cuts in ([307], [300, 4] + [1] * 3, [17] * 18 + [1], [16, 1, 15, 32, 31, 2, 63, 64, 65] + [1] * 18, [257, 50], [256, 2, 49]):
            s = r.admit()
            check(feed(r, s, toks, cuts), want, dtype, f"far tokens {name} {dtype} cuts {cuts[:3]}")
            r.release(s)


def test_first_tokens_and_long_decoding(folders):
    d, (cfg, W) = folders("other", CONFIGS["other"], seed=7)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=192)
        for n in (1, 2, 3, 4, 6):
            toks = helpers.random_tokens(cfg["vocab"], n, seed=20 + n)
            for cuts in ([1] * n, [n]):
                s = r.admit()
                check(feed(r, s, toks, cuts), oracle(cfg, W, toks), dtype, f"{n} first tokens in {cuts} ({dtype})")
                r.release(s)
        toks = helpers.random_tokens(cfg["vocab"], 183, seed=33)
        s = r.admit()
        check(feed(r, s, toks, [3] + [1] * 180), oracle(cfg, W, toks), dtype, f"long decoding ({dtype})")
        r.release(s)


def test_a_slot_used_again_starts_from_nothing(folders):
    """A request's keys and state must not reach the request that gets its slot and pages next."""
    d, (cfg, W) = folders("far_looped", FAR["looped"], seed=9, touch=slow)
    a, b = helpers.random_tokens(2000, 60, seed=61), helpers.random_tokens(2000, 40, seed=62)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_seqs=1, max_tokens=64)
        s = r.admit()
        feed(r, s, a, [30] + [1] * 30)
        r.release(s)
        assert r.admit() == s
        check(feed(r, s, b, [25] + [1] * 15), oracle(cfg, W, b), dtype, f"the slot's second request ({dtype})")
        r.release(s)


def test_captured_steps_equal_uncaptured_ones_and_side_by_side_equals_in_turn(folders):
    """Steps replayed from CUDA graphs give the bits of steps launched kernel by kernel, and the feed-forward on a stream of
    its own beside the mixer those of the two in turn."""
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("wide", CONFIGS["wide"], seed=7)
    toks = [helpers.random_tokens(cfg["vocab"], 100, seed=70 + i) for i in range(3)]
    outs = []
    for graphs, beside in ((True, True), (False, True), (True, False), (False, False)):
        r = runner_for(d, "bfloat16", max_tokens=128, cuda_graphs=graphs)
        for b in r.model.blocks:
            b.overlap = beside
        slots = [r.admit() for _ in toks]
        got = []
        for lo, hi in ((0, 12), (12, 24), (24, 36), (36, 48)):       # the same shape again and again: captured, then replayed
            got.append(r.step([StepEntry(s, t[lo:hi], [hi - lo - 1]) for s, t in zip(slots, toks)]).cpu())
        for i in range(48, 100):
            got.append(r.step([StepEntry(s, [t[i]], [0]) for s, t in zip(slots, toks)]).cpu())
        outs.append(torch.cat(got))
        if graphs:
            assert r.graph_replays > 0
        assert any(b.mixer.defers(3) for b in r.model.blocks)        # the wide model's few-row steps do hand back partial sums
    for o in outs[1:]:
        assert torch.equal(outs[0], o)


def test_long_prompts_on_the_tensor_core_attention(folders):
    """Steps of some hundred rows on the bfloat16 path take the tiled attention kernels and the products on pairs of SMs: a
    prompt of 700 tokens whole, in portions beside a second request, and decoded on, against the plain implementation."""
    from cajeta_llm_b200.engine.step import StepEntry
    d, (cfg, W) = folders("wide", CONFIGS["wide"], seed=7)
    toks = helpers.random_tokens(cfg["vocab"], 700, seed=12)
    other = helpers.random_tokens(cfg["vocab"], 40, seed=13)
    want, want_other = oracle(cfg, W, toks), oracle(cfg, W, other)
    for dtype in ("bfloat16", "float32"):
        r = runner_for(d, dtype, max_tokens=768, max_seqs=2)
        s = r.admit()
        check(feed(r, s, toks, [700]), want, dtype, f"700 tokens whole ({dtype})")
        r.release(s)
        s, s2 = r.admit(), r.admit()
        got, got2, at = [], [], 0
        for n, m in ((300, 17), (256, 1), (130, 22), (1, 0), (1, 0), (12, 0)):
            entries = [StepEntry(s, toks[at:at + n], list(range(n)))]
            lo = sum(g.shape[0] for g in got2)
            if m:
                entries.append(StepEntry(s2, other[lo:lo + m], list(range(m))))
            out = r.step(entries).cpu()
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
    wa, wb = oracle(cfg, W, a), oracle(cfg, W, b)
    got = {n: torch.from_numpy(np.fromfile(os.path.join(str(tmp_path), f"{n}.f32"), dtype="<f4").reshape(-1, cfg["vocab"])) for n in range(3)}
    check(got[0], wa[10:11], "float32", "step 0")
    check(got[1], wb[8:9], "float32", "step 1")
    check(got[2], wa[[11, 19]], "float32", "step 2")


def random_config(seed):
    """A configuration drawn at random: layer order, every size and constant, the looped stretch."""
    rng = random.Random(seed)
    width = rng.choice([40, 72, 136, 256])
    big = width >= 128
    layers = []
    for _ in range(rng.randint(1, 5)):
        ff = rng.choice([None, rng.randint(8, 80), 256 if big else 64])
        if rng.random() < 0.6:
            kv = rng.randint(1, 3)
            dim = rng.choice([32, 64, 96, 128, 72]) if big and rng.random() < 0.6 else rng.randint(2, 24)
            vdim = dim if rng.random() < 0.5 else rng.choice([32, 64, 128, rng.randint(1, 40)])
            layers.append(attn(heads=kv * rng.randint(1, 4), kv_heads=kv, dim=dim, vdim=vdim, dims=2 * rng.randint(1, dim // 2),
                               base=rng.choice([100.0, 10000.0, 500000.0]), scale=rng.choice([0.1, 0.3, 1.0 / math.sqrt(dim)]),
                               softcap=rng.choice([2.0, 15.0, 50.0]), ff=ff))
        else:
            layers.append(gru(width=rng.choice([128, 152]) if big and rng.random() < 0.5 else rng.randint(1, 90), ff=ff))
    loop = None
    if rng.random() < 0.7:
        start = rng.randint(0, len(layers) - 1)
        loop = (start, rng.randint(start + 1, len(layers)), rng.randint(1, 3))
    return config_of(layers, width=width, vocab=rng.choice([70, 131, 300]), eps=rng.choice([1e-5, 1e-6]), mult=rng.choice([0.25, 0.5, 0.37, 1.0]), loop=loop)


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(folders, seed):
    raw = random_config(7000 + seed)
    d, (cfg, W) = folders(f"random{seed}", raw, seed=100 + seed)
    toks = helpers.random_tokens(cfg["vocab"], 120, seed=seed)
    want = oracle(cfg, W, toks)
    for dtype in ("float32", "bfloat16"):
        r = runner_for(d, dtype, max_tokens=128)
        for cuts in ([120], [17, 2, 9, 60] + [1] * 32):
            s = r.admit()
            check(feed(r, s, toks, cuts), want, dtype, f"{json.dumps(raw)} {dtype} cuts {cuts[:3]}")
            r.release(s)


def test_a_second_norm_that_nothing_reads_may_be_in_the_file(folders, tmp_path):
    """A layer without a feed-forward: its second norm's weight is neither asked for nor refused."""
    from cajeta_llm_b200.weights.safetensors_io import Checkpoint, write_safetensors
    d, (cfg, W) = folders("mingru", ALONE["mingru"], seed=3)
    ck = Checkpoint(d)
    tensors = {n: ck.load(n) for n in ck.names()}
    ck.close()
    assert "l0.norm2" not in tensors
    tensors["l0.norm2"] = torch.full((48,), 7.0, dtype=torch.bfloat16)
    write_safetensors(str(tmp_path / "model.safetensors"), tensors)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    toks = helpers.random_tokens(90, 20, seed=1)
    r = runner_for(str(tmp_path), "float32", max_tokens=32)
    check(feed(r, r.admit(), toks, [20]), oracle(cfg, W, toks), "float32", "with the idle norm")


# -- the kernels against formulas ----------------------------------------------------------------------------
def _scan_formula(x, W, state):
    """One request's rows [n, 3W] in float64 from ``state``: outputs [n, W] and the state after them."""
    x = x.double()
    z, u, g = x[:, :W], x[:, W:2 * W], x[:, 2 * W:]
    z = torch.sigmoid(z)
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S, out = state.double(), []
    for t in range(x.shape[0]):
        S = (1 - z[t]) * S + z[t] * c[t]
        out.append(S * g[t] * torch.sigmoid(g[t]))
    return torch.stack(out) if out else torch.empty((0, W), dtype=torch.float64), S


@pytest.mark.parametrize("width", [1, 5, 24, 130, 2504])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_scan_against_the_formula(width, dtype):
    """Requests of every length around the tiles' edges beside one another, one that brings no rows, gates near 0 and near 1,
    a state carried over from an earlier step."""
    from cajeta_llm_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(width)
    for lens in ([1, 2, 16, 17, 0, 255, 256, 257], [700], [33, 1, 1, 600]) if width < 2000 else ([300, 1, 17],):
        R, T = len(lens), sum(lens)
        x = torch.randn((T, 3 * width), generator=g)
        x[:, :width] = x[:, :width] * 4 - 4                       # gates: mostly nearly shut, some open
        x[: T // 3, :width] += 40.0 * (torch.rand((T // 3, width), generator=g) < 0.02)      # some wide open, far out
        x[:, width:2 * width] *= 3
        x[0, 2 * width:] = -200.0                                 # silu of a large negative number
        state = torch.randn((R + 3, width + 7), generator=g)
        slots = torch.randperm(R + 3, generator=g)[:R].int()
        starts = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
        want, want_state = [], state.clone()
        for i, n in enumerate(lens):
            o, s = _scan_formula(x[int(starts[i]):int(starts[i + 1])], width, state[int(slots[i]), 3:3 + width])
            want.append(o)
            want_state[int(slots[i]), 3:3 + width] = s.float()
        dev_state, out = state.to(DEV), torch.empty((T, width), dtype=dtype, device=DEV)
        filler = torch.cat([slots, torch.tensor([-1], dtype=torch.int32)])          # a request a step's layout is filled up with
        K.gated_scan(x.to(DEV), 0, width, 2 * width, width, dev_state, 3, torch.cat([starts, starts[-1:]]).to(DEV), filler.to(DEV), R + 1, out)
        w = torch.cat(want)
        tol = 2e-5 if dtype == torch.float32 else 1e-2
        assert float(((out.cpu().double() - w).abs() / (w.abs() + 0.05)).max()) < tol
        assert float((dev_state.cpu() - want_state).abs().max()) < 2e-5
    # single tokens of many requests
    R = 37
    x, state = torch.randn((R, 3 * width), generator=g), torch.randn((R, width), generator=g)
    dev_state, out = state.to(DEV), torch.empty((R, width), dtype=dtype, device=DEV)
    K.gated_scan(x.to(DEV), 0, width, 2 * width, width, dev_state, 0, torch.arange(R + 1, dtype=torch.int32, device=DEV),
                 torch.arange(R, dtype=torch.int32, device=DEV), R, out, single=True)
    for i in range(R):
        o, s = _scan_formula(x[i:i + 1], width, state[i])
        assert float((dev_state[i].cpu().double() - s).abs().max()) < 1e-5
        assert float(((out[i].cpu().double() - o[0]).abs() / (o[0].abs() + 0.05)).max()) < (2e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("rows,width", [(1, 5), (3, 48), (7, 1026), (300, 2048), (260, 4096), (2, 8192), (3, 9000)])
def test_two_norms_of_one_row(rows, width):
    from cajeta_llm_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(rows)
    x, wa, wb = torch.randn((rows, width), generator=g), torch.randn(width, generator=g), torch.randn(width, generator=g)
    pa, pb = torch.randn((3, rows, width), generator=g), torch.randn((2, rows, width), generator=g)
    for parts in ((), (pa,), (pa, pb)):
        for dtype in (torch.float32, torch.bfloat16):
            xd = x.to(DEV)
            a, b = torch.empty((rows, width), dtype=dtype, device=DEV), torch.empty((rows, width), dtype=dtype, device=DEV)
            K.rmsnorm_pair(xd, wa.to(DEV), wb.to(DEV), 1e-5, a, b, partials=tuple(p.to(DEV) for p in parts))
            s = x.double() + sum((p.double().sum(0) for p in parts), torch.zeros_like(x, dtype=torch.float64))
            y = s / torch.sqrt(s.pow(2).mean(-1, keepdim=True) + 1e-5)
            tol = 1e-5 if dtype == torch.float32 else 1e-2
            assert float((xd.cpu().double() - s).abs().max()) < 1e-5
            for got, w in ((a, wa), (b, wb)):
                want = y * w.double()
                assert float(((got.cpu().double() - want).abs() / (want.abs() + 1.0)).max()) < tol
    hs = x.to(DEV)
    K.add_partials(hs, pa.to(DEV), pb.to(DEV))
    assert float((hs.cpu().double() - (x.double() + pa.double().sum(0) + pb.double().sum(0))).abs().max()) < 1e-5


@pytest.mark.parametrize("heads,kv,hd,vd,rot", [(4, 2, 128, 128, 64), (3, 1, 96, 96, 20), (2, 2, 12, 10, 6), (5, 1, 7, 9, 2), (2, 1, 200, 260, 100), (3, 3, 64, 32, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_heads_normed_without_a_weight_rotated_in_pairs(heads, kv, hd, vd, rot, dtype):
    """Rotation first and the norm after it, as written down, against the kernel's one pass (which norms before it rotates)."""
    from cajeta_llm_b200.csrc import kernels as K
    g = torch.Generator().manual_seed(hd)
    T, page, eps = 37, 16, 1e-5
    C = (heads + kv) * hd + kv * vd
    x = torch.randn((T, C), generator=g) * 2
    x[3] *= 1e-3                                                  # eps counts in this row
    pos = torch.randint(0, 5000, (T,), generator=g).int()
    inv = (1000.0 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)).float()
    table = torch.arange(T, dtype=torch.int32)[:, None].repeat(1, 5000 // page + 1).contiguous()      # request t's every page is page t
    q = torch.empty((T, heads, hd), dtype=dtype, device=DEV)
    kp, vp = torch.zeros((T, kv, page, hd), dtype=dtype, device=DEV), torch.zeros((T, kv, page, vd), dtype=dtype, device=DEV)
    K.head_prepare(x.to(DEV), 0, heads * hd, (heads + kv) * hd, q, kp, vp, pos.to(DEV), torch.arange(T, dtype=torch.int32, device=DEV), table.to(DEV),
                   page, heads, kv, hd, vd, rot, inv.to(DEV), 1.0, None, None, eps, True, unit_qk=True, unit_v=True, pairs=True)

    def ready(rows, t):
        out = rows.double().clone()
        for i in range(rot // 2):
            a = float(torch.tensor(float(pos[t])) * inv[i])
            u, w = rows[:, 2 * i].double(), rows[:, 2 * i + 1].double()
            out[:, 2 * i], out[:, 2 * i + 1] = u * math.cos(a) - w * math.sin(a), w * math.cos(a) + u * math.sin(a)
        return out / torch.sqrt(out.pow(2).mean(-1, keepdim=True) + eps)

    tol = 1e-5 if dtype == torch.float32 else 2e-2
    for t in range(T):
        p = int(pos[t]) % page
        v = x[t, (heads + kv) * hd:].view(kv, vd).double()
        assert float((q[t].cpu().double() - ready(x[t, :heads * hd].view(heads, hd), t)).abs().max()) < tol
        assert float((kp[t, :, p].cpu().double() - ready(x[t, heads * hd:(heads + kv) * hd].view(kv, hd), t)).abs().max()) < tol
        assert float((vp[t, :, p].cpu().double() - v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)).abs().max()) < tol


def _attention_case(heads, kv, hd, vd, lens, priors, seed, unit=True):
    """Planes, tables and queries of requests with ``priors`` cached keys that bring ``lens`` rows; everything bfloat16."""
    g = torch.Generator().manual_seed(seed)
    page = 16
    need = [-(-(p + n) // page) for p, n in zip(priors, lens)]
    order = torch.randperm(sum(need) + 3, generator=g).int()
    table = torch.full((len(lens), max(need)), -1, dtype=torch.int32)
    at = 0
    for i, n in enumerate(need):
        table[i, :n] = order[at:at + n]
        at += n
    kp, vp = torch.randn((sum(need) + 3, kv, page, hd), generator=g), torch.randn((sum(need) + 3, kv, page, vd), generator=g)
    q = torch.randn((sum(lens), heads, hd), generator=g)
    if unit:
        q, kp = (t / t.pow(2).mean(-1, keepdim=True).sqrt() for t in (q, kp))
    pos = torch.cat([torch.arange(p, p + n) for p, n in zip(priors, lens)]).int()
    req = torch.cat([torch.full((n,), i) for i, n in enumerate(lens)]).int()
    starts = torch.tensor([0] + list(np.cumsum(lens)), dtype=torch.int32)
    return tuple(t.to(DEV) for t in (q.bfloat16(), kp.bfloat16(), vp.bfloat16(), table, pos, req, starts, torch.tensor(priors, dtype=torch.int32)))


def _attention_formula(q, kp, vp, table, pos, req, scale, cap, sink):
    q, kp, vp = (t.cpu().double() for t in (q, kp, vp))
    table, pos, req = table.cpu(), pos.cpu(), req.cpu()
    heads, kv = q.shape[1], kp.shape[1]
    out = torch.zeros((q.shape[0], heads, vp.shape[-1]), dtype=torch.float64)
    for t in range(q.shape[0]):
        keys = torch.arange(int(pos[t]) + 1)
        pages = table[int(req[t]), keys // 16].long()
        k, v = kp[pages, :, keys % 16], vp[pages, :, keys % 16]                     # [n, kv, .]
        k, v = k.repeat_interleave(heads // kv, 1), v.repeat_interleave(heads // kv, 1)
        s = torch.einsum("hd,nhd->hn", q[t], k) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        m = torch.maximum(s.max(-1, keepdim=True).values, torch.tensor(sink if sink is not None else -1e30))
        e = torch.exp(s - m)
        d = e.sum(-1, keepdim=True) + (torch.exp(sink - m) if sink is not None else 0.0)
        out[t] = torch.einsum("hn,nhd->hd", e / d, v)
    return out


SIZES = [(4, 2, 128, 128), (9, 3, 96, 96), (8, 2, 64, 64), (3, 3, 32, 32), (4, 2, 40, 72), (2, 1, 104, 24), (12, 1, 8, 128)]


@pytest.mark.parametrize("heads,kv,hd,vd", SIZES)
def test_capped_attention_with_a_constant_sink(heads, kv, hd, vd):
    """Every attention kernel of the general path, prompt portions and single tokens, against the formula: no sink, one of
    score 0, one that outweighs the keys, one far below them; capped and not; values of another size than keys."""
    from cajeta_llm_b200.csrc import kernels as K
    lens, priors = [70, 1, 2, 33, 1], [0, 0, 15, 300, 129]
    q, kp, vp, table, pos, req, starts, prior = _attention_case(heads, kv, hd, vd, lens, priors, seed=hd)
    ones = [200, 1, 129, 128, 520]
    dq, dkp, dvp, dtable, dpos, dreq, _, _ = _attention_case(heads, kv, hd, vd, [1] * 5, [n - 1 for n in ones], seed=hd + 1)
    scale = 2.0 / math.sqrt(hd)
    scratch = K.DecodeScratch()
    for cap, sink in ((0.0, None), (9.0, 0.0), (30.0, 5.0), (2.0, 0.0), (50.0, -30.0), (0.0, 0.0)):
        given = K.NO_SINK if sink is None else sink
        want, dwant = _attention_formula(q, kp, vp, table, pos, req, scale, cap, sink), _attention_formula(dq, dkp, dvp, dtable, dpos, dreq, scale, cap, sink)

        def close(out, w, what, tol=0.02):
            err = float((out.cpu().double() - w).abs().max())
            assert err < tol * max(1.0, float(w.abs().max())), f"{what} cap {cap} sink {sink}: off by {err:.4f}"

        out = torch.empty((q.shape[0], heads, vd), dtype=torch.bfloat16, device=DEV)
        K.paged_attention(q, out, kp, vp, pos, req, table, 16, heads, kv, hd, 0, scale, value_dim=vd, softcap=cap, sink=given)
        close(out, want, "row by row")
        for rows in (64, 128):
            out.fill_(7.0)
            K.prefill_attention(q, out, kp, vp, starts, prior, table, 16, heads, kv, hd, 0, scale, block_rows=rows, softcap=cap, sink=given, value_dim=vd)
            close(out, want, f"tiles of {rows} rows")
        dout = torch.empty((5, heads, vd), dtype=torch.bfloat16, device=DEV)
        for later in (False, True):
            dout.fill_(7.0)
            K.decode_attention(dq, dout, dkp, dvp, dpos, dreq, dtable, 16, heads, kv, hd, 0, scale, max(ones), scratch, tensor_cores=True,
                               merge_later=later, softcap=cap, sink=given, value_dim=vd)
            close(dout, dwant, f"decode, merged {'later' if later else 'by the last block'}")
        if hd == vd == 128:
            for exact in (False, True):
                # the bound on the scores decides between the exact forms: 22.6 here (unit heads), or unknown
                for bound in ((0.0,) if not exact else (0.0, scale * hd * 1.02)):
                    for rows in (128, 256):
                        out.fill_(7.0)
                        K.prefill_attention_tc(q, out, kp, vp, starts, prior, table, 16, heads, kv, hd, 0, scale, block_rows=rows, softcap=cap,
                                               sink=given, exact_cap=exact, score_bound=bound)
                        close(out, want, f"tcgen05, exact {exact}, bound {bound}")


@pytest.mark.parametrize("cap", [38.0, 60.0, 120.0, 10.0])
def test_exact_forms_of_the_cap_agree(cap):
    """The polynomial forms (three to five terms, by the scores' bound over the cap) and the exponential one give the same
    attention to float32 rounding of the scores; keys aligned with the queries so that scores reach their bound."""
    from cajeta_llm_b200.csrc import kernels as K
    heads, hd = 2, 128
    q, kp, vp, table, pos, req, starts, prior = _attention_case(heads, 1, hd, hd, [200], [0], seed=5)
    kp[table[0, 3].long(), 0, 5] = q[180, 0]                      # one score at its bound
    kp[table[0, 7].long(), 0, 1] = -q[190, 1]                     # and one at minus its bound
    scale = 2.0 / math.sqrt(hd)
    bound = scale * hd * 1.02                                     # 23.1: 0.61, 0.38 and 0.19 of the first three caps, beyond the last
    want = _attention_formula(q, kp, vp, table, pos, req, scale, cap, 0.0)
    outs = []
    for b in (bound, 0.0):
        out = torch.empty((200, heads, hd), dtype=torch.bfloat16, device=DEV)
        K.prefill_attention_tc(q, out, kp, vp, starts, prior, table, 16, heads, 1, hd, 0, scale, softcap=cap, sink=0.0, exact_cap=True, score_bound=b)
        outs.append(out.cpu().double())
        assert float((outs[-1] - want).abs().max()) < 0.02
    # the same weights but for a rounding of bfloat16 here and there
    assert float((outs[0] - outs[1]).abs().max()) < 0.02 and float(((outs[0] - outs[1]).abs() > 1e-3).double().mean()) < 0.02


@pytest.mark.parametrize("rows", [3, 40, 200, 600])
def test_scaled_results_of_the_products(rows):
    """``out_scale`` multiplies sum and bias as they are stored or added: every product kernel, and partial sums."""
    from cajeta_llm_b200.csrc import kernels as K
    from cajeta_llm_b200.parts.base import Runtime
    from cajeta_llm_b200.parts.linear import project, project_split, splits_few_rows
    g = torch.Generator().manual_seed(rows)
    for dtype, k, n in (("float32", 70, 90), ("bfloat16", 40, 50), ("bfloat16", 1024, 256), ("bfloat16", 1024, 520)):
        rt = Runtime(dtype, DEV)
        x, w, b = torch.randn((rows, k), generator=g), torch.randn((n, k), generator=g) / math.sqrt(k), torch.randn(n, generator=g)
        x, w = rt.matrix(x), rt.matrix(w)
        base = torch.randn((rows, n), generator=g)
        want = 0.37 * (x.cpu().double() @ w.cpu().double().T + b.double())
        out = base.to(DEV)
        project(rt, x, w, out, bias=b.to(DEV), accumulate=True, out_scale=0.37)
        assert float((out.cpu().double() - base.double() - want).abs().max()) < 2e-5
        project(rt, x, w, out, bias=b.to(DEV), out_scale=0.37)
        assert float((out.cpu().double() - want).abs().max()) < 2e-5
        parts = project_split(rt, x, w, bias=b.to(DEV), out_scale=0.37)
        assert (parts is not None) == splits_few_rows(rt, rows, w)
        if parts is not None:
            assert float((parts.sum(0).cpu().double() - want).abs().max()) < 2e-5
    with pytest.raises(ValueError):
        project(rt, x, w, torch.empty((rows, n), dtype=torch.bfloat16, device=DEV), out_scale=2.0)
    with pytest.raises(K.KernelError):
        K.gemm_tc(x, w, torch.empty((rows, n), dtype=torch.bfloat16, device=DEV), K.EPI_STORE_BF16, True, 16, out_scale=2.0)
