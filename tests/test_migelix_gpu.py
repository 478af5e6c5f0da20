"""Migelix through the engine against the plain implementation (tests/plain_migelix.py, float64).

Four small models that differ in every size and option (tests/migelix_models.py) are run whole, as a prompt followed by
single tokens, in portions down to two tokens, and as mixed batches in a pool whose pages and slots are used again;
single mechanisms are isolated by one-layer configurations; weights are bent where random ones would hide a fault (a far
key, the sink, a cap, the edges of a window, a state that must still hold its first token).

Bounds.  The measure is the RMS over the vocabulary of the logits' difference (mean taken off) over the RMS of the
wanted logits, the largest over the rows.  What rounding alone does depends on the model, so it is measured: the plain
implementation is run once more in float32, or with the operands and results of its products rounded to bfloat16 values, and
the engine may be three times as far from the exact logits as that run is (or 2e-4 and 2e-2, where that is more).  Where a test
rests on a mechanism mattering, it checks that with the plain implementation first.
"""
import copy

import numpy as np
import pytest
import torch

import plain_migelix as plain
from migelix_models import CONFIGS, _config, attention, delta, heads_of, layer, make_weights, parallel, rel_error, wkv, write_model

pytestmark = pytest.mark.gpu

AT_LEAST = {"float32": 2e-4, "bfloat16": 2e-2}
DTYPES = ["float32", "bfloat16"]
_cache = {}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, model folder)."""
    base = tmp_path_factory.mktemp("migelix")
    out = {}
    for i, (name, cfg) in enumerate(sorted(CONFIGS.items())):
        w = make_weights(cfg, seed=800 + i)
        out[name] = (cfg, w, write_model(cfg, w, str(base / name)))
    return out


def _engine(model_dir, dtype, max_tokens=512, page_size=16, max_requests=4):
    from sandyrt_b200.engine.step import Engine
    from sandyrt_b200.models.model import load_model

    model = load_model(model_dir, device="cuda:0", dtype=getattr(torch, dtype))
    eng = Engine(model, max_tokens=max_tokens, page_size=page_size, max_requests=max_requests)
    eng.cache.device_caches.poison()
    return eng


def _tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


def _want(cfg, w, ids):
    key = (id(w), tuple(ids))
    if key not in _cache:
        _cache[key] = [plain.forward(cfg, w, ids).numpy(), {}, w]        # w kept alive: its id is the key
    return _cache[key][0]


def _bound(cfg, w, ids, dtype):
    want = _want(cfg, w, ids)
    rounding = _cache[(id(w), tuple(ids))][1]
    if dtype not in rounding:
        run = plain.forward_rounded(cfg, w, ids) if dtype == "bfloat16" else plain.forward(cfg, w, ids, dtype=torch.float32)
        rounding[dtype] = rel_error(run.numpy(), want)
    return max(AT_LEAST[dtype], 3 * rounding[dtype])


def _run_cuts(eng, rid, ids, cuts, release=True):
    from sandyrt_b200.engine.step import StepEntry

    rows, pos = [], 0
    for n in cuts:
        rows.append(eng.step([StepEntry(rid, ids[pos:pos + n], list(range(n)))]).cpu().numpy().copy())
        pos += n
    assert pos == len(ids)
    eng.check_status()
    if release:
        eng.release(rid)
    return np.concatenate(rows, axis=0)


def _check(got, model, ids, dtype, what):
    cfg, w = model
    e, bound = rel_error(got, _want(cfg, w, ids)), _bound(cfg, w, ids, dtype)
    assert e < bound, f"{what}: relative error {e:.3e} (bound {bound:.1e})"


# ---- whole models under every way of cutting the work -------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompts_and_first_tokens(models, name, dtype):
    cfg, w, path = models[name]
    eng = _engine(path, dtype)
    for i, n in enumerate([1, 2, 5, 33, 150, 300]):
        ids = _tokens(cfg, n, seed=i)
        _check(_run_cuts(eng, f"r{i}", ids, [n]), (cfg, w), ids, dtype, f"{name}: whole prompt of {n}")
    eng.cache.alloc.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_then_single_tokens(models, name, dtype):
    """Most of the request in one step, the last 60 tokens one by one (the later ones replay a recorded graph)."""
    cfg, w, path = models[name]
    eng = _engine(path, dtype)
    ids = _tokens(cfg, 161, seed=7)
    got = _run_cuts(eng, "r", ids, [101] + [1] * 60)
    _check(got, (cfg, w), ids, dtype, f"{name}: prompt + 60 single tokens")
    assert eng.graph_replays > 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_of_changing_size(models, name, dtype):
    """Portions below and above the size from which the recurrences work in chunks, through parts of chunks, page borders
    and the windows' edges, down to two tokens."""
    cfg, w, path = models[name]
    eng = _engine(path, dtype)
    ids = _tokens(cfg, 131, seed=11)
    for cuts in ([24, 24, 24, 24, 35], [2, 3, 17, 16, 15, 31, 2, 13, 32], [1, 2, 1, 3, 124], [64, 67], [16, 16, 32, 1, 1, 65],
                 [23, 2, 14, 2, 7, 1, 23, 59], [47, 1, 2, 14, 1, 66], [8, 8, 9, 7, 99], [33, 65, 33], [2] * 65 + [1]):
        assert sum(cuts) == len(ids)
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"{name}: portions {cuts[:9]}")
    eng.cache.alloc.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_first_tokens_in_every_division(models, name, dtype):
    cfg, w, path = models[name]
    eng = _engine(path, dtype)
    ids = _tokens(cfg, 6, seed=13)
    for cuts in ([1] * 6, [2, 2, 2], [1, 5], [5, 1], [3, 1, 2], [6]):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"{name}: first tokens as {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(models, name, dtype):
    """Up to four live requests, portions of some beside single tokens of others; the pool holds 12 pages of 16 tokens
    for requests that need 31 in all, pages poisoned.  Each request's rows must equal what it gives alone (its states sit
    in a slot that other requests held before)."""
    from sandyrt_b200.engine.step import StepEntry

    cfg, w, path = models[name]
    eng = _engine(path, dtype, max_tokens=192, page_size=16, max_requests=4)
    lengths = [37, 90, 21, 64, 45, 30, 118, 17]
    prompts = [_tokens(cfg, n, seed=20 + i) for i, n in enumerate(lengths)]
    rng = np.random.default_rng(1)
    fed = [0] * len(prompts)
    got = [[] for _ in prompts]
    live, nxt, slots_seen = [], 0, []
    while nxt < len(prompts) or live:
        while nxt < len(prompts) and len(live) < 4:
            if sum(-(-lengths[r] // 16) for r in live) + -(-lengths[nxt] // 16) > 12:
                break
            live.append(nxt)
            nxt += 1
        entries = []
        for r in live:
            left = lengths[r] - fed[r]
            n = int(rng.integers(2, min(left, 41) + 1)) if left > 8 and rng.random() < 0.6 else 1
            entries.append(StepEntry(r, prompts[r][fed[r]:fed[r] + n], list(range(n))))
        if rng.random() < 0.3 and len(entries) > 1:
            entries.pop(int(rng.integers(0, len(entries))))
        out = eng.step(entries).cpu().numpy()
        row = 0
        for e in entries:
            n = len(e.tokens)
            got[e.rid].append(out[row:row + n].copy())
            row += n
            fed[e.rid] += n
            slots_seen.append((e.rid, eng.cache.alloc.slot(e.rid)))
        for r in list(live):
            if fed[r] == lengths[r]:
                eng.release(r)
                live.remove(r)
        eng.cache.alloc.check()
    eng.check_status()
    assert len({s for _, s in slots_seen}) <= 4 and len({r for r, _ in slots_seen}) == 8      # slots were used again
    for r, ids in enumerate(prompts):
        _check(np.concatenate(got[r], axis=0), (cfg, w), ids, dtype, f"{name}: mixed request {r}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_a_batch_gives_each_request_what_it_gives_alone(models, name, dtype):
    """Unequal requests in one step against each alone: same rows, beyond rounding."""
    from sandyrt_b200.engine.step import StepEntry

    cfg, w, path = models[name]
    eng = _engine(path, dtype)
    prompts = [_tokens(cfg, n, seed=40 + n) for n in (110, 3, 29, 1)]
    alone = [_run_cuts(eng, f"a{i}", p, [len(p)]) for i, p in enumerate(prompts)]
    out = eng.step([StepEntry(f"b{i}", p, list(range(len(p)))) for i, p in enumerate(prompts)]).cpu().numpy()
    row = 0
    for i, p in enumerate(prompts):
        e = rel_error(out[row:row + len(p)], alone[i])
        assert e < (1e-5 if dtype == "float32" else 2e-2), f"request {i} in a batch differs from itself alone by {e:.2e}"
        row += len(p)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_across_pages_and_windows(models, name, dtype):
    """300 single tokens behind a short prompt, pages of 8: every page border and every window's edge is crossed by a
    decoded token, and the pages behind the windows go back to the pool (the request holds few of them at its end)."""
    cfg, w, path = models[name]
    eng = _engine(path, dtype, max_tokens=512, page_size=8)
    ids = _tokens(cfg, 310, seed=3)
    got = _run_cuts(eng, "r", ids, [10] + [1] * 300, release=False)
    _check(got, (cfg, w), ids, dtype, f"{name}: 300 decoded tokens")
    groups = eng.cache.layout.groups
    assert groups
    for g in range(len(groups)):
        held = sum(1 for b in eng.cache.alloc.block_list("r", g) if b >= 0)
        assert held <= -(-groups[g].spec.window // 8) + 2
    eng.release("r")


def test_a_pool_smaller_than_the_request(models):
    """A request of 400 tokens through windows of 24 and 17 in a pool of 160 tokens: pages come round again and again, with
    another request beside it."""
    from sandyrt_b200.engine.step import StepEntry

    cfg, w, path = models["A"]
    eng = _engine(path, "float32", max_tokens=160, page_size=8)
    ids, other = _tokens(cfg, 400, seed=4), _tokens(cfg, 30, seed=5)
    got, pos, fed, beside = [], 0, 0, []
    for n in [30, 20, 2, 1, 1, 40, 17] + [1, 2, 30] * 8 + [1] * 25:
        entries = [StepEntry("r", ids[pos:pos + n], list(range(n)))]
        if fed < 30:
            entries.append(StepEntry("o", other[fed:fed + 2], [0, 1]))
            fed += 2
        out = eng.step(entries).cpu().numpy().copy()
        got.append(out[:n])
        beside.append(out[n:])
        pos += n
        eng.cache.alloc.check()
    assert pos == 400
    eng.check_status()
    _check(np.concatenate(got), (cfg, w), ids, "float32", "400 tokens in a pool of 160")
    _check(np.concatenate(beside), (cfg, w), other, "float32", "the request beside it")


# ---- single mechanisms --------------------------------------------------------------------------------
def _one_model(tmp_path, cfg, seed, bend=None):
    w = make_weights(cfg, seed)
    if bend:
        bend(w)
        w = {k: v.to(torch.bfloat16).to(torch.float32) for k, v in w.items()}
    return w, write_model(cfg, w, str(tmp_path / f"m{seed}"))


def _without(cfg, w, ids, change_cfg=None, change_w=None, sink=True):
    """Logits of the plain implementation with one thing changed, to show that the thing matters."""
    cfg2, w2 = copy.deepcopy(cfg), dict(w)
    if change_cfg:
        change_cfg(cfg2)
    if change_w:
        change_w(w2)
    return plain.forward(cfg2, w2, ids, sink=sink).numpy()


SMALL = dict(left=lambda **kw: heads_of(2, 1, 16, size=20, rot=8, **kw), right=lambda: delta(2, 2, 8, 8))
ONE_LAYER = {
    "attention, no window, no rotation": lambda: [layer(attention(3, 1, 24), None)],
    "attention, no cap": lambda: [layer(attention(4, 2, 48, size=20, rot=48, softcap=None), None)],
    "attention, a window of one token": lambda: [layer(attention(2, 1, 16, size=1), None)],
    "attention, one head of one entry": lambda: [layer(attention(1, 1, 1, size=7, scale=2.0), None)],
    "attention, heads of 200": lambda: [layer(attention(2, 1, 200, size=30, rot=10), None)],
    "attention, sixteen heads on one": lambda: [layer(attention(16, 1, 64, size=50, rot=16), None)],
    "attention, heads of 128": lambda: [layer(attention(6, 2, 128, size=37, rot=48), None)],
    "left side alone": lambda: [layer(parallel(heads_of(6, 3, 32, size=13, rot=20, base=40.0, yarn=(3.0, 20, 6.0, 0.5)), delta(1, 1, 4, 4), 1.5, 0.0), None)],
    "left side alone, heads of 128, all of an entry turned": lambda: [layer(parallel(heads_of(8, 1, 128, rot=128, base=1e5, yarn=(16.0, 64, 32.0, 1.0)), delta(1, 1, 4, 4), 1.0, 0.0), None)],
    "left side alone, a ramp of no length": lambda: [layer(parallel(heads_of(2, 2, 16, rot=16, base=10.0, yarn=(2.0, 9, 3.0, 3.0)), delta(1, 1, 4, 4), 1.0, 0.0), None)],
    "delta rule": lambda: [layer(parallel(SMALL["left"](), delta(6, 2, 20, 24, conv=4, rank=5, gate_rank=9), 0.0, 1.0), None)],
    "delta rule, one channel": lambda: [layer(parallel(SMALL["left"](), delta(2, 1, 1, 1, conv=2, rank=1, gate_rank=1), 0.0, 2.0), None)],
    "delta rule, wide": lambda: [layer(parallel(SMALL["left"](), delta(1, 1, 200, 136, conv=8, rank=40, gate_rank=33), 0.0, -0.7), None)],
    "delta rule, heads of 128": lambda: [layer(parallel(SMALL["left"](), delta(2, 1, 128, 128, conv=4, rank=24, gate_rank=8), 0.0, 1.0), None)],
    "delta rule, one tap": lambda: [layer(parallel(SMALL["left"](), delta(3, 3, 16, 20, conv=1, rank=3, gate_rank=5), 0.0, 1.0), None)],
    "time mixing": lambda: [layer(wkv(3, 20, rank=5), None)],
    "time mixing, one channel": lambda: [layer(wkv(2, 1, rank=1), None)],
    "time mixing, wide": lambda: [layer(wkv(1, 200, rank=40), None)],
    "time mixing, heads of 64": lambda: [layer(wkv(3, 64, rank=16), None)],
    "a feed-forward": lambda: [layer(wkv(1, 8), 100)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mechanism_alone(tmp_path, which, dtype):
    cfg = _config(61, 48, ONE_LAYER[which](), cap=None)
    w, path = _one_model(tmp_path, cfg, seed=5)
    eng = _engine(path, dtype)
    ids = _tokens(cfg, 110, seed=1)
    _check(_run_cuts(eng, "r", ids, [110]), (cfg, w), ids, dtype, f"{which}, whole")
    _check(_run_cuts(eng, "r", ids, [40, 2, 35, 8, 1] + [1] * 24), (cfg, w), ids, dtype, f"{which}, in portions")


def _sharp(w, pre="l0.mix.", by=4.0):
    w[pre + "q"] = by * w[pre + "q"]


def _attending(kind, dim, heads=4, kv=2, **kw):
    """One layer of attention: by itself with a cap too high to matter, or as the left side of a parallel mixer."""
    if kind == "single":
        return layer(attention(heads, kv, dim, softcap=200.0, **kw), None), "l0.mix."
    return layer(parallel(heads_of(heads, kv, dim, **kw), delta(1, 1, 8, 8), 1.0, 0.0), None), "l0.mix.left."


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,dim", [("single", 16), ("single", 64), ("left", 24), ("left", 64), ("left", 128)])
def test_a_windows_edge_decides(tmp_path, kind, dim, dtype):
    """Sharp scores, a window of 21 and 300 tokens: a window one token off moves the logits (the plain implementation shows
    it).  Whole, in portions and decoded, in pages of 16 and of 8."""
    l, pre = _attending(kind, dim, size=21, rot=8, base=100.0)
    cfg = _config(53, 64, [l], cap=None)
    w, path = _one_model(tmp_path, cfg, seed=9, bend=lambda w: _sharp(w, pre))
    ids = _tokens(cfg, 300, seed=2)
    want = _want(cfg, w, ids)
    for size in (20, 22):
        def other(c):
            m = c["layers"][0]["mixer"]
            (m if kind == "single" else m["left"])["mask"]["size"] = size
        assert rel_error(_without(cfg, w, ids, change_cfg=other)[-200:], want[-200:]) > 0.1, size
    for page in (16, 8):
        eng = _engine(path, dtype, max_tokens=512, page_size=page)
        _check(_run_cuts(eng, "r", ids, [300]), (cfg, w), ids, dtype, "window, whole")
        _check(_run_cuts(eng, "r", ids, [150, 2, 98, 18] + [1] * 32), (cfg, w), ids, dtype, "window, portions and single tokens")
        _check(_run_cuts(eng, "r", ids, [3] + [1] * 297), (cfg, w), ids, dtype, "window, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,dim", [("single", 32), ("single", 64), ("left", 64), ("left", 128)])
def test_a_far_key_among_hundreds(tmp_path, kind, dim, dtype):
    """No window, sharp scores over 400 tokens: a key that is lost or off by one moves the logits."""
    l, pre = _attending(kind, dim, rot=4, base=1e6)
    cfg = _config(53, 64, [l], cap=None)
    w, path = _one_model(tmp_path, cfg, seed=10, bend=lambda w: _sharp(w, pre, 6.0))
    ids = _tokens(cfg, 400, seed=2)

    def near(c):
        m = c["layers"][0]["mixer"]
        (m if kind == "single" else m["left"])["mask"] = {"size": 200}

    assert rel_error(_without(cfg, w, ids, change_cfg=near)[-32:], _want(cfg, w, ids)[-32:]) > 0.1
    eng = _engine(path, dtype, max_tokens=512)
    _check(_run_cuts(eng, "r", ids, [400]), (cfg, w), ids, dtype, "sharp scores, whole")
    _check(_run_cuts(eng, "r", ids, [250, 100, 18] + [1] * 32), (cfg, w), ids, dtype, "sharp scores, portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64, 128])
def test_the_sink_decides(tmp_path, dim, dtype):
    """Sinks of their own for every head, some far above the scores, some far below: without them, or with one for all, the
    logits move."""
    cfg = _config(53, 64, [layer(parallel(heads_of(4, 2, dim, size=30, rot=8), delta(1, 1, 8, 8), 1.0, 0.0), None)], cap=None)

    def bend(w):
        w["l0.mix.left.sink"] = torch.tensor([6.0, -8.0, 3.0, 1.0])

    w, path = _one_model(tmp_path, cfg, seed=12, bend=bend)
    ids = _tokens(cfg, 90, seed=6)
    assert rel_error(_without(cfg, w, ids, sink=False), _want(cfg, w, ids)) > 0.2
    assert rel_error(_without(cfg, w, ids, change_w=lambda w2: w2.update({"l0.mix.left.sink": torch.zeros(4)})), _want(cfg, w, ids)) > 0.2
    eng = _engine(path, dtype)
    _check(_run_cuts(eng, "r", ids, [90]), (cfg, w), ids, dtype, "sinks, whole")
    _check(_run_cuts(eng, "r", ids, [1, 1, 40, 3] + [1] * 45), (cfg, w), ids, dtype, "sinks, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [24, 64, 128])
def test_the_caps_decide(tmp_path, dim, dtype):
    """Scores and logits far beyond their caps: another cap, or none, gives other logits; the window and the gate beside it."""
    cfg = _config(53, 64, [layer(attention(4, 2, dim, size=40, rot=8, softcap=3.0), None)], cap=4.0)
    w, path = _one_model(tmp_path, cfg, seed=13, bend=lambda w: (_sharp(w, by=8.0), w.update(embed=4.0 * w["embed"])))
    ids = _tokens(cfg, 130, seed=6)
    want = _want(cfg, w, ids)
    assert rel_error(_without(cfg, w, ids, change_cfg=lambda c: c["layers"][0]["mixer"].update(softcap=6.0)), want) > 0.05
    assert rel_error(_without(cfg, w, ids, change_cfg=lambda c: c.update(logit_softcap=8.0)), want) > 0.05
    eng = _engine(path, dtype)
    _check(_run_cuts(eng, "r", ids, [130]), (cfg, w), ids, dtype, "caps, whole")
    _check(_run_cuts(eng, "r", ids, [60, 2, 20] + [1] * 48), (cfg, w), ids, dtype, "caps, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_rescaled_rotation_decides(tmp_path, dtype):
    """Frequencies of which some are kept, some slowed and some in between: each constant of the rescaling moves the logits,
    and so does its magnitude."""
    yarn = (4.0, 40, 4.0, 0.5)
    cfg = _config(53, 64, [layer(parallel(heads_of(4, 2, 64, size=60, rot=48, base=200.0, yarn=yarn), delta(1, 1, 8, 8), 1.0, 0.0), None)], cap=None)
    w, path = _one_model(tmp_path, cfg, seed=14, bend=lambda w: _sharp(w, "l0.mix.left."))
    ids = _tokens(cfg, 140, seed=6)
    for key, value in (("factor", 8.0), ("original", 90), ("fast", 1.5), ("slow", 2.0)):
        def other(c):
            c["layers"][0]["mixer"]["left"]["rot"]["scaling"][key] = value
        assert rel_error(_without(cfg, w, ids, change_cfg=other)[-40:], _want(cfg, w, ids)[-40:]) > 0.05, key
    eng = _engine(path, dtype)
    _check(_run_cuts(eng, "r", ids, [140]), (cfg, w), ids, dtype, "rescaled rotation, whole")
    _check(_run_cuts(eng, "r", ids, [60, 2, 30] + [1] * 48), (cfg, w), ids, dtype, "rescaled rotation, decoded")


def _recurrent(kind):
    if kind == "wkv":
        return _config(53, 48, [layer(wkv(4, 32, rank=3), None)], cap=None)
    return _config(53, 48, [layer(parallel(SMALL["left"](), delta(4, 2, 32, 16, conv=4, rank=3, gate_rank=4), 0.0, 1.0), None)], cap=None)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["wkv", "delta"])
def test_a_state_that_still_holds_its_first_tokens(tmp_path, kind, dtype):
    """A recurrence alone that hardly fades: what the first tokens wrote is still much of the state after 200, so a state
    that is lost between steps, starts from another request's numbers or is cleared late shows.  Run beside another
    request, then again in the slot the other one left."""
    from sandyrt_b200.engine.step import StepEntry

    cfg = _recurrent(kind)

    def slow(w):
        if kind == "wkv":
            w["l0.mix.w0"] = torch.full((128,), -7.0)
        else:
            w["l0.mix.right.A_log"] = torch.full((4,), -6.0)
            w["l0.mix.right.b"] = 0.2 * w["l0.mix.right.b"]

    w, path = _one_model(tmp_path, cfg, seed=15, bend=slow)
    ids = _tokens(cfg, 220, seed=5)
    want = _want(cfg, w, ids)
    cut = plain.forward(cfg, w, ids[20:]).numpy()
    assert rel_error(cut[-10:], want[-10:]) > 0.02          # the first 20 tokens still matter 200 tokens later
    eng = _engine(path, dtype, max_tokens=768, max_requests=2)
    other = _tokens(cfg, 90, seed=6)
    got, pos = [], 0
    eng.step([StepEntry("other", other[:50], [])])
    for n in [30, 2, 1, 80, 7] + [1] * 100:
        entries = [StepEntry("r", ids[pos:pos + n], list(range(n)))]
        if pos < 40:
            entries.append(StepEntry("other", other[50 + pos:50 + pos + 1], []))
        got.append(eng.step(entries).cpu().numpy()[:n].copy())
        pos += n
    assert pos == 220
    eng.check_status()
    _check(np.concatenate(got), (cfg, w), ids, dtype, "long memory beside another request")
    eng.release("other")
    eng.release("r")
    _check(_run_cuts(eng, "again", ids, [219, 1]), (cfg, w), ids, dtype, "long memory in a slot used before")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["wkv", "delta"])
def test_channels_fade_each_at_its_own_pace(tmp_path, kind, dtype):
    """Decays from none to everything in one token, channel by channel: one pace for all of a head's channels gives other
    logits, and running sums of logarithms in the hundreds must not overflow."""
    cfg = _recurrent(kind)
    name = "l0.mix.w0" if kind == "wkv" else "l0.mix.right.dt_bias"
    lo, hi = (-8.0, 6.0) if kind == "wkv" else (-9.0, 40.0)

    def spread(w):
        n = w[name].numel()
        w[name] = torch.linspace(lo, hi, n)[torch.randperm(n, generator=torch.Generator().manual_seed(1))]

    w, path = _one_model(tmp_path, cfg, seed=16, bend=spread)
    ids = _tokens(cfg, 150, seed=5)
    assert rel_error(_without(cfg, w, ids, change_w=lambda w2: w2.update({name: torch.full_like(w[name], -2.0)})), _want(cfg, w, ids)) > 0.1
    eng = _engine(path, dtype)
    for cuts in ([150], [1] * 150, [9, 40, 2, 33, 31, 35], [32, 64, 54]):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"paces, {cuts[:5]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_token_before_and_the_bonus_decide(tmp_path, dtype):
    """Mixes close to one (every projection reads mostly the token before) and large bonuses: the last input of a step must
    reach the next one, and the bonus the current token alone."""
    cfg = _config(53, 72, [layer(wkv(3, 24, rank=3), None), layer(wkv(2, 40, rank=2), 40)], cap=None)

    def bend(w):
        for i in (0, 1):
            for k, s in enumerate("rkvgw"):
                w[f"l{i}.mix.mu.{s}"] = torch.full((72,), 0.95 - 0.1 * k)
            w[f"l{i}.mix.u"] = 3.0 * w[f"l{i}.mix.u"]

    w, path = _one_model(tmp_path, cfg, seed=18, bend=bend)
    ids = _tokens(cfg, 120, seed=5)
    want = _want(cfg, w, ids)
    assert rel_error(_without(cfg, w, ids, change_w=lambda w2: w2.update({"l1.mix.u": torch.zeros(2, 40)})), want) > 0.1
    swapped = lambda w2: w2.update({"l0.mix.mu.r": w["l0.mix.mu.w"], "l0.mix.mu.w": w["l0.mix.mu.r"]})
    assert rel_error(_without(cfg, w, ids, change_w=swapped), want) > 0.05
    eng = _engine(path, dtype)
    for cuts in ([120], [1] * 120, [7, 40, 2, 33, 38], [2] * 60):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"token before, {cuts[:5]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_convolutions_that_reach_far_back(tmp_path, dtype):
    """Eight taps of which the first decides, in portions shorter than the taps and in single tokens."""
    cfg = _config(53, 48, [layer(parallel(SMALL["left"](), delta(4, 2, 16, 16, conv=8, rank=3, gate_rank=4), 0.0, 1.0), None)], cap=None)

    def bend(w):
        for s in "qkv":
            t = 0.2 * w[f"l0.mix.right.{s}.conv"]
            t[:, 0] += 1.5
            w[f"l0.mix.right.{s}.conv"] = t

    w, path = _one_model(tmp_path, cfg, seed=19, bend=bend)
    ids = _tokens(cfg, 90, seed=5)
    eng = _engine(path, dtype)
    for cuts in ([90], [1] * 90, [2, 3, 1, 4, 5, 2, 40, 33], [8, 7, 75]):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"taps, {cuts[:5]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_layers_on_one_set_of_tensors_keep_caches_of_their_own(tmp_path, dtype):
    """Each kind of layer three times on the same tensors: one shared cache or state would give other logits from the second
    token on."""
    cfg = _config(53, 64, [layer(parallel(heads_of(4, 2, 32, size=19, rot=16), delta(2, 1, 16, 24)), None), layer(wkv(3, 24), 40),
                           layer(attention(2, 1, 64, size=25, rot=16), None)], reuse=(0, 1, 2, 1, 0, 2))
    w, path = _one_model(tmp_path, cfg, seed=21)
    ids = _tokens(cfg, 130, seed=8)
    eng = _engine(path, dtype)
    _check(_run_cuts(eng, "r", ids, [130]), (cfg, w), ids, dtype, "shared tensors, whole")
    _check(_run_cuts(eng, "r", ids, [50, 20, 2, 28] + [1] * 30), (cfg, w), ids, dtype, "shared tensors, in portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_through_many_key_tiles(tmp_path, dtype):
    """900 tokens through heads of 64 (the tcgen05 prompt kernel) and of 128 and 48 (mma.sync) with windows of a few hundred;
    portions that start inside tiles; then single tokens."""
    cfg = _config(97, 128, [layer(attention(2, 1, 64, size=300, rot=64, softcap=15.0), None), layer(wkv(2, 64, rank=8), None),
                            layer(parallel(heads_of(4, 1, 128, size=257, rot=64), delta(2, 2, 64, 64, rank=8, gate_rank=8)), None),
                            layer(attention(3, 3, 48, rot=16, softcap=15.0), None)])
    w, path = _one_model(tmp_path, cfg, seed=31, bend=lambda w: (_sharp(w, "l0.mix.", 3.0), _sharp(w, "l2.mix.left.", 3.0), _sharp(w, "l3.mix.", 3.0)))
    eng = _engine(path, dtype, max_tokens=1024)
    ids = _tokens(cfg, 900, seed=2)
    _check(_run_cuts(eng, "r", ids, [900]), (cfg, w), ids, dtype, "long prompt, whole")
    _check(_run_cuts(eng, "r", ids, [330, 2, 409, 130] + [1] * 29), (cfg, w), ids, dtype, "long prompt, portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_delta_rule_as_a_mixer_of_its_own(dtype):
    """The kind that is no side of another mixer, alone, in three steps of two requests, against the plain mixer."""
    from sandyrt_b200.models.spec import PartSpec
    from sandyrt_b200.parts.harness import PartHarness

    c = dict(heads=4, kv_heads=2, dim=16, vdim=24, conv=4)
    names = {"q": "q", "k": "k", "v": "v", "o": "o", "norm": "norm", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv", "beta": "b",
             "decay_in": "a1", "decay_out": "a2", "dt_bias": "dt_bias", "a_log": "A_log", "gate_in": "g1", "gate_out": "g2"}
    spec = PartSpec("channel_delta", {"width": 40, "eps": 1e-5, "n_heads": 4, "n_qk_heads": 2, "qk_dim": 16, "v_dim": 24, "conv_taps": 4,
                                      "rank": 5, "gate_rank": 3}, {n: n for n in names})
    part = PartHarness("mixer", spec, getattr(torch, dtype), seed=4)
    w = {names[k]: torch.from_numpy(v).double() for k, v in part.tensors().items()}
    g = torch.Generator().manual_seed(3)
    lens, fed = (61, 23), [0, 0]
    hs = [torch.randn(n, 40, generator=g).mul(6).to(getattr(torch, dtype)) for n in lens]
    want = [plain.delta_mixer(c, w, "", h.double(), 1e-5) for h in hs]
    for step in ((40, 2), (20, 20), (1, 1)):
        h = torch.cat([hs[i][fed[i]:fed[i] + n] for i, n in enumerate(step)]).cuda()
        x = torch.zeros(h.shape[0], 40, device="cuda")
        part.set_step([(fed[i], n) for i, n in enumerate(step)])
        part.run_mixer(h, x)
        torch.cuda.synchronize()
        ref = torch.cat([want[i][fed[i]:fed[i] + n] for i, n in enumerate(step)])
        fed = [f + n for f, n in zip(fed, step)]
        size = ref.pow(2).mean().sqrt().item()
        assert (x.double().cpu() - ref).pow(2).mean().sqrt().item() < (1e-5 if dtype == "float32" else 2e-2) * size, step


# ---- the entry point --------------------------------------------------------------------------------------
def test_greedy_generation_through_the_entry_point(models):
    """LLM.generate (scheduler, prompt portions, decode bursts) on three requests at once, float32: the same tokens as
    greedy decoding with the plain implementation, wherever its top two logits are clearly apart."""
    from sandyrt_b200.engine.llm import LLM

    cfg, w, path = models["A"]
    llm = LLM(path, dtype="float32", cache_tokens=1024, max_live=4, prefill_chunk_tokens=24, max_step_tokens=64)
    prompts = [_tokens(cfg, n, seed=60 + n) for n in (5, 40, 71)]
    outs = llm.generate(prompts, max_tokens=20)
    for p, r in zip(prompts, outs):
        assert r.finish_reason == "length" and len(r.output_ids) == 20
        ids = list(p)
        for tok in r.output_ids:
            l = _want(cfg, w, ids)[-1]
            top2 = np.sort(l)[-2:]
            if top2[1] - top2[0] > 1e-3:
                assert tok == int(np.argmax(l)), f"token {len(ids) - len(p)} of the request with {len(p)} prompt tokens"
            ids.append(tok)


@pytest.mark.parametrize("name,shape", [("l0.mix.right.a2", (8, 4)), ("l0.mix.right.g2", (8, 5))])
def test_matrices_that_do_not_fit_together_are_refused(tmp_path, name, shape):
    """The two matrices of a low-rank product take their rank from the weight file and must agree on it."""
    from sandyrt_b200.errors import ConfigError
    from sandyrt_b200.models.model import load_model

    cfg = _config(31, 16, [layer(parallel(SMALL["left"](), delta(1, 1, 8, 8, rank=3, gate_rank=3)), None)])
    w = make_weights(cfg, seed=1)
    w[name] = torch.zeros(*shape)
    with pytest.raises(ConfigError, match="rank"):
        load_model(write_model(cfg, w, str(tmp_path / "m")), device="cuda:0", dtype=torch.float32)
