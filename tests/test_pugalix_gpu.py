"""Pugalix through the engine against the plain implementation (tests/plain_pugalix.py, float64).

Four small models that differ in every size and option (tests/pugalix_models.py) are run whole, as a prompt followed by
single tokens, in portions down to two tokens, and as mixed batches in a pool whose pages and slots are used again;
single mechanisms are isolated by one-layer configurations; weights are bent where random ones would hide a fault (a far
kept key, the one in the softmax's denominator, the edges of a window, a state that must still hold its first token).

Bounds.  The measure is the RMS over the vocabulary of the logits' difference (mean taken off) over the RMS of the
wanted logits, the largest over the rows.  What rounding alone does depends on the model (a head of a matrix memory whose
first read-outs nearly vanish is divided by its own tiny root mean square, which lifts the last bits: up to 7e-4 in float32
with some small heads), so it is measured: the plain implementation is run once more in float32, or with the operands and
results of its products rounded to bfloat16 values, and the engine may be three times as far from the exact logits as
that run is (or 2e-4 and 2e-2, where that is more).  Where a test rests on a mechanism
mattering, it checks that with the plain implementation first.
"""
import copy

import numpy as np
import pytest
import torch

import plain_pugalix as plain
from pugalix_models import CONFIGS, _config, attention, gla, layer, make_weights, mlstm, rel_error, write_model

pytestmark = pytest.mark.gpu

AT_LEAST = {"float32": 2e-4, "bfloat16": 2e-2}
DTYPES = ["float32", "bfloat16"]
_cache = {}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, model folder)."""
    base = tmp_path_factory.mktemp("pugalix")
    out = {}
    for i, (name, cfg) in enumerate(sorted(CONFIGS.items())):
        w = make_weights(cfg, seed=700 + i)
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
    for s, g in zip([s for s in eng.model.cache_specs() if s["kind"] == "paged"], range(99)):
        held = sum(1 for b in eng.cache.alloc.block_list("r", g) if b >= 0)
        assert held <= -(-s["keep_first"] // 8) + -(-s["window"] // 8) + 2
    eng.release("r")


def test_a_pool_smaller_than_the_request(models):
    """A request of 400 tokens through windows of 24 and 40 in a pool of 160 tokens: its kept pages stay, the others come
    round again and again, with another request beside it."""
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


ONE_LAYER = {
    "attention, no window, no rotation": lambda: [layer(attention(3, 1, 24, 40), None)],
    "attention, keys wider than values": lambda: [layer(attention(4, 2, 48, 16, size=20, keep=3, rot=48), None)],
    "attention, more kept tokens than the window is long": lambda: [layer(attention(2, 2, 32, 32, size=5, keep=37, rot=2), None)],
    "attention, a window of one token": lambda: [layer(attention(2, 1, 16, 16, size=1, keep=0), None)],
    "attention, one head of one entry": lambda: [layer(attention(1, 1, 1, 1, size=7, keep=1, scale=2.0), None)],
    "attention, heads of 200": lambda: [layer(attention(2, 1, 200, 136, size=30, keep=4, rot=10), None)],
    "attention, sixteen heads on one": lambda: [layer(attention(16, 1, 64, 64, size=50, keep=6, rot=16), None)],
    "gated linear attention": lambda: [layer(gla(3, 20, 24, tau=8.0, rank=5), None)],
    "gated linear attention, one channel": lambda: [layer(gla(2, 1, 1, tau=1.0, rank=1), None)],
    "gated linear attention, wide": lambda: [layer(gla(1, 200, 136, tau=32.0, rank=40), None)],
    "gated linear attention, fast fading": lambda: [layer(gla(2, 32, 16, tau=0.25, rank=3), None)],
    "matrix memory": lambda: [layer(mlstm(3, 24, 20, cap=3.0), None)],
    "matrix memory, wide": lambda: [layer(mlstm(1, 136, 72, cap=15.0), None)],
    "a reader of another layer's keys": lambda: [layer(attention(4, 2, 16, 24, size=12, keep=2, rot=8), None),
                                                 layer(attention(4, 2, 16, 24, size=31, keep=9, rot=8, kv_from=0), None)],
    "a feed-forward": lambda: [layer(gla(1, 8, 8), 100)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", sorted(ONE_LAYER))
def test_each_mechanism_alone(tmp_path, which, dtype):
    cfg = _config(61, 48, ONE_LAYER[which](), scale=1.3)
    w, path = _one_model(tmp_path, cfg, seed=5)
    eng = _engine(path, dtype)
    ids = _tokens(cfg, 110, seed=1)
    _check(_run_cuts(eng, "r", ids, [110]), (cfg, w), ids, dtype, f"{which}, whole")
    _check(_run_cuts(eng, "r", ids, [40, 2, 35, 8, 1] + [1] * 24), (cfg, w), ids, dtype, f"{which}, in portions")


def _sharp(w, layer=0, by=4.0):
    w[f"l{layer}.mix.q"] = by * w[f"l{layer}.mix.q"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [16, 64])
def test_far_kept_keys_decide(tmp_path, dim, dtype):
    """Sharp scores, a short window, 9 kept tokens (they end inside the first page of 16, and inside the second page of 8)
    and 400 tokens: one kept token more or fewer, or a window one off, moves the logits (the plain implementation shows
    it).  Whole, in portions and decoded."""
    cfg = _config(53, 64, [layer(attention(4, 2, dim, dim, size=20, keep=9, rot=8, base=100.0), None)])
    w, path = _one_model(tmp_path, cfg, seed=9, bend=_sharp)
    ids = _tokens(cfg, 400, seed=2)
    want = _want(cfg, w, ids)
    mask = lambda **kw: (lambda c: c["layers"][0]["mixer"]["mask"].update(**kw))
    for kw in (dict(keep_first=8), dict(keep_first=10), dict(size=19), dict(size=21), dict(keep_first=0)):
        assert rel_error(_without(cfg, w, ids, change_cfg=mask(**kw))[-32:], want[-32:]) > 0.1, kw
    for page in (16, 8):
        eng = _engine(path, dtype, max_tokens=512, page_size=page)
        _check(_run_cuts(eng, "r", ids, [400]), (cfg, w), ids, dtype, "kept keys, whole")
        _check(_run_cuts(eng, "r", ids, [250, 2, 98, 18] + [1] * 32), (cfg, w), ids, dtype, "kept keys, portions and single tokens")
        _check(_run_cuts(eng, "r", ids, [3] + [1] * 397), (cfg, w), ids, dtype, "kept keys, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [32, 64])
def test_a_far_key_among_hundreds(tmp_path, dim, dtype):
    """No window, sharp scores over 400 tokens: a key that is lost or off by one moves the logits."""
    cfg = _config(53, 64, [layer(attention(4, 2, dim, dim, rot=4, base=1e6), None)])
    w, path = _one_model(tmp_path, cfg, seed=10, bend=lambda w: _sharp(w, by=6.0))
    ids = _tokens(cfg, 400, seed=2)
    assert rel_error(_without(cfg, w, ids, change_cfg=lambda c: c["layers"][0]["mixer"].update(mask={"size": 200, "keep_first": 0}))[-32:],
                     _want(cfg, w, ids)[-32:]) > 0.1
    eng = _engine(path, dtype, max_tokens=512)
    _check(_run_cuts(eng, "r", ids, [400]), (cfg, w), ids, dtype, "sharp scores, whole")
    _check(_run_cuts(eng, "r", ids, [250, 100, 18] + [1] * 32), (cfg, w), ids, dtype, "sharp scores, portions and single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_one_in_the_denominator_decides(tmp_path, dtype):
    """Scores pulled far below zero by the biases of q and k: the heads see almost nothing but the one, and the plain
    softmax would see everything (the plain implementation shows it)."""
    cfg = _config(53, 64, [layer(attention(4, 2, 16, 16, size=30, keep=4, scale=0.25), None)])

    def bend(w):
        w["l0.mix.q.b"] = torch.ones(64)
        w["l0.mix.k.b"] = -torch.ones(32)

    w, path = _one_model(tmp_path, cfg, seed=12, bend=bend)
    ids = _tokens(cfg, 90, seed=6)
    assert rel_error(_without(cfg, w, ids, sink=False), _want(cfg, w, ids)) > 0.2
    eng = _engine(path, dtype)
    _check(_run_cuts(eng, "r", ids, [90]), (cfg, w), ids, dtype, "the one, whole")
    _check(_run_cuts(eng, "r", ids, [1, 1, 40, 3] + [1] * 45), (cfg, w), ids, dtype, "the one, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["gla", "mlstm"])
def test_a_state_that_still_holds_its_first_tokens(tmp_path, kind, dtype):
    """A recurrence alone that hardly fades: what the first tokens wrote is still much of the state after 200, so a state
    that is lost between steps, starts from another request's numbers or is cleared late shows.  Run beside another
    request, then again in the slot the other one left."""
    from sandyrt_b200.engine.step import StepEntry

    cfg = _config(53, 48, [layer(gla(4, 32, 16, tau=64.0, rank=3) if kind == "gla" else mlstm(4, 32, 16, cap=20.0), None)])

    def slow(w):
        if kind == "gla":
            w["l0.mix.a2.b"] = torch.full((128,), 6.0)
        else:
            w["l0.mix.f.b"] = torch.full((4,), 9.0)
            w["l0.mix.f"] = 0.1 * w["l0.mix.f"]

    w, path = _one_model(tmp_path, cfg, seed=15, bend=slow)
    ids = _tokens(cfg, 220, seed=5)
    want = _want(cfg, w, ids)
    cut = plain.forward(cfg, w, ids[20:]).numpy()
    assert rel_error(cut[-10:], want[-10:]) > 0.05          # the first 20 tokens still matter 200 tokens later
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
def test_channels_fade_each_at_its_own_pace(tmp_path, dtype):
    """Decays from none to everything in one token, channel by channel (the biases spread over -20 .. 20, tau 1): one pace
    for all of a head's channels, or the decay on the value's side, gives other logits, and running sums of logarithms in
    the hundreds must not overflow."""
    cfg = _config(53, 48, [layer(gla(2, 40, 24, tau=1.0, rank=6), None)])

    def spread(w):
        w["l0.mix.a2.b"] = torch.linspace(-20, 20, 80)[torch.randperm(80, generator=torch.Generator().manual_seed(1))]

    w, path = _one_model(tmp_path, cfg, seed=16, bend=spread)
    ids = _tokens(cfg, 150, seed=5)

    def one_pace(w2):
        w2["l0.mix.a2.b"] = torch.zeros(80)

    assert rel_error(_without(cfg, w, ids, change_w=one_pace), _want(cfg, w, ids)) > 0.2
    eng = _engine(path, dtype)
    for cuts in ([150], [1] * 150, [9, 40, 2, 33, 31, 35], [32, 64, 54]):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"paces, {cuts[:5]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_input_gates_that_reach_their_cap(tmp_path, dtype):
    """Large gate pre-activations: the caps decide, the running maximum rises and falls, and a small cap is not a large one."""
    cfg = _config(53, 48, [layer(mlstm(3, 16, 24, cap=4.0), None)])

    def loud(w):
        for k in ("i", "f"):
            w[f"l0.mix.{k}"] = 8.0 * w[f"l0.mix.{k}"]

    w, path = _one_model(tmp_path, cfg, seed=17, bend=loud)
    ids = _tokens(cfg, 120, seed=5)
    assert rel_error(_without(cfg, w, ids, change_cfg=lambda c: c["layers"][0]["mixer"].update(gate_cap=30.0)), _want(cfg, w, ids)) > 0.05
    eng = _engine(path, dtype)
    for cuts in ([120], [1] * 120, [7, 40, 2, 33, 38]):
        _check(_run_cuts(eng, "r", ids, cuts), (cfg, w), ids, dtype, f"capped gates, {cuts[:5]}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_reader_sees_further_than_the_layer_it_reads(tmp_path, dtype):
    """The layer that writes looks back 10 positions, the one that reads 60 and 12 kept ones (and the other way round):
    the pages stay as long as either needs them.  Sharp scores in the reader."""
    for k, (a, b) in enumerate((((10, 0), (60, 12)), ((60, 12), (10, 0)), ((10, 3), (0, 0)))):
        cfg = _config(53, 64, [layer(attention(4, 2, 64, 64, size=a[0], keep=a[1], rot=16), None), layer(gla(1, 16, 16), None),
                               layer(attention(4, 2, 64, 64, size=b[0], keep=b[1], rot=16, kv_from=0), None)])
        w, path = _one_model(tmp_path, cfg, seed=20 + k, bend=lambda w: _sharp(w, layer=2))
        ids = _tokens(cfg, 260, seed=8)
        eng = _engine(path, dtype, max_tokens=320, page_size=8)
        _check(_run_cuts(eng, "r", ids, [260]), (cfg, w), ids, dtype, f"reader {k}, whole")
        _check(_run_cuts(eng, "r", ids, [90, 70, 2, 38] + [1] * 60), (cfg, w), ids, dtype, f"reader {k}, in portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_through_many_key_tiles(tmp_path, dtype):
    """900 tokens through heads of 64 (the tcgen05 prompt kernel) and of 48 (mma.sync) with windows of a few hundred and
    kept tokens in several tiles; portions that start inside tiles; then single tokens."""
    cfg = _config(97, 128, [layer(attention(2, 1, 64, 64, size=300, keep=140, rot=64), None), layer(gla(2, 64, 64), None),
                            layer(attention(3, 3, 40, 48, size=257, keep=65, rot=16), None), layer(mlstm(2, 64, 64), None)])
    w, path = _one_model(tmp_path, cfg, seed=31, bend=lambda w: (_sharp(w, 0, 3.0), _sharp(w, 2, 3.0)))
    eng = _engine(path, dtype, max_tokens=1024)
    ids = _tokens(cfg, 900, seed=2)
    _check(_run_cuts(eng, "r", ids, [900]), (cfg, w), ids, dtype, "long prompt, whole")
    _check(_run_cuts(eng, "r", ids, [330, 2, 409, 130] + [1] * 29), (cfg, w), ids, dtype, "long prompt, portions and single tokens")


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


def test_matrices_that_do_not_fit_together_are_refused(tmp_path):
    """The decay's two matrices take their rank from the weight file and must agree on it."""
    from sandyrt_b200.errors import ConfigError
    from sandyrt_b200.models.model import load_model

    cfg = _config(31, 16, [layer(gla(1, 8, 8, rank=3), None)])
    w = make_weights(cfg, seed=1)
    w["l0.mix.a2"] = torch.zeros(8, 4)
    with pytest.raises(ConfigError, match="rank"):
        load_model(write_model(cfg, w, str(tmp_path / "m")), device="cuda:0", dtype=torch.float32)
