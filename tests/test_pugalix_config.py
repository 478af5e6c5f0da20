"""Pugalix without a GPU: the configuration and its checks, the model description (parts, run order, shared cache
entries, tensor names), pages that a window gives back and kept first ones, and properties of the plain implementation
that the GPU tests lean on."""
import copy
import math

import pytest
import torch

import plain_pugalix as plain
from pugalix_models import CONFIGS, _config, attention, gla, layer, make_weights, mlstm, tensor_shapes

from sandyrt_b200.config.base import ConfigError, config_from_normalised
from sandyrt_b200.config.pugalix import PugalixConfig


def _without_rank(raw):
    raw = copy.deepcopy(raw)
    for l in raw["layers"]:
        l["mixer"].pop("rank", None)
    return raw


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_description_names_every_tensor_with_its_shape(name):
    from sandyrt_b200.models.model import build_model

    cfg = config_from_normalised(CONFIGS[name])
    assert isinstance(cfg, PugalixConfig) and cfg.vocab_size == CONFIGS[name]["vocab"]
    cfg.validate()
    got = {k: list(v.shape) for k, v in build_model(cfg).tensor_requests().items()}
    assert got == tensor_shapes(CONFIGS[name])
    # the decay's rank is the weight file's where the configuration is silent
    got = {k: list(v.shape) for k, v in build_model(config_from_normalised(_without_rank(CONFIGS[name]))).tensor_requests().items()}
    want = tensor_shapes(CONFIGS[name])
    for k, v in want.items():
        if k.endswith(".a1"):
            assert got[k] == [-1, v[1]]
        elif k.endswith(".a2"):
            assert got[k] == [v[0], -1]
        else:
            assert got[k] == v


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_run_order_and_cache_entries(name):
    """A layer with kv_from works on the other layer's cache entry and writes nothing; every other layer has its own."""
    from sandyrt_b200.models.model import describe

    raw = CONFIGS[name]
    spec = describe(config_from_normalised(raw))
    assert [c.layer for c in spec.schedule] == list(range(len(raw["layers"])))
    entry, nxt = {}, 0
    for c, l, s in zip(spec.schedule, raw["layers"], spec.layers):
        src = l["mixer"].get("kv_from")
        if src is None:
            assert c.cache == nxt and c.write_cache
            nxt += 1
        else:
            assert c.cache == entry[src] and not c.write_cache
        entry[c.layer] = c.cache
        assert s.block == "pre_norm" and sorted(s.norms) == (["feed_forward", "mixer"] if l["mlp"] else ["mixer"])
        assert s.mixer.kind == {"attention": "windowed_attention", "gla": "gated_linear_attention", "mlstm": "matrix_memory"}[l["type"]]
        assert s.feed_forward.kind == ("gated_mlp" if l["mlp"] else "none")
    assert spec.n_caches() == nxt and spec.max_positions is None
    assert spec.embedding.params["scale"] == raw["embedding"]["scale"] and spec.head.params["tied"] is False


def test_config_round_trip_and_constants_reach_the_parts():
    from sandyrt_b200.models.model import describe

    raw = CONFIGS["A"]
    cfg = PugalixConfig.from_dict(raw)
    assert PugalixConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict()["layers"] == raw["layers"] and cfg.to_dict()["embedding"] == raw["embedding"]
    spec = describe(cfg)
    m, src = spec.layers[0].mixer.params, raw["layers"][0]["mixer"]
    assert (m["n_heads"], m["n_kv_heads"], m["qk_dim"], m["v_dim"]) == (src["heads"], src["kv_heads"], src["dim"], src["vdim"])
    assert (m["window"], m["keep_first"], m["rot_dims"], m["rot_base"]) == (24, 5, 8, 1000.0) and m["scale"] == src["scale"]
    assert m["rot_interleaved"] and m["unit_sink"] and m["out_gate"] and m["bias"] and m["own_kv"]
    r = spec.layers[3].mixer.params
    assert (r["window"], r["keep_first"]) == (40, 2) and not r["own_kv"]
    assert "k" not in spec.layers[3].mixer.tensors and "v_bias" not in spec.layers[3].mixer.tensors
    assert spec.layers[4].mixer.params["tau"] == 4.0 and spec.layers[2].mixer.params["gate_cap"] == 12.0
    assert spec.layers[4].mixer.params["eps"] == raw["norm"]["eps"]


def test_optional_keys_have_their_defaults():
    raw = _config(31, 16, [layer(attention(2, 2, 8, 8), None)])
    del raw["embedding"], raw["layers"][0]["mixer"]["kv_heads"]
    raw["layers"][0]["mixer"].update(mask=None, rot=None, kv_from=None)
    cfg = config_from_normalised(raw)
    cfg.validate()
    assert cfg.to_dict()["embedding"] == {"scale": 1.0} and cfg.to_dict()["layers"][0]["mixer"]["kv_heads"] == 2


BAD = {
    "no width": lambda c: c.pop("width"),
    "no layers": lambda c: c.update(layers=[]),
    "an unknown layer type": lambda c: c["layers"][0].update(type="lstm"),
    "heads that do not divide": lambda c: c["layers"][0]["mixer"].update(kv_heads=3),
    "an odd number of rotated entries": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    "more rotated entries than a head has": lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18),
    "a negative window": lambda c: c["layers"][0]["mixer"]["mask"].update(size=-1),
    "keys of a later layer": lambda c: c["layers"][3]["mixer"].update(kv_from=4),
    "keys of a recurrence": lambda c: c["layers"][3]["mixer"].update(kv_from=1),
    "keys of other sizes": lambda c: c["layers"][3]["mixer"].update(dim=8),
    "keys of a reader": lambda c: c["layers"].append(layer(attention(4, 2, 16, 32, kv_from=3), None)),
    "a tau of zero": lambda c: c["layers"][1]["mixer"].update(tau=0.0),
    "a gate cap of zero": lambda c: c["layers"][2]["mixer"].update(gate_cap=0.0),
    "a state beyond the kernels": lambda c: c["layers"][1]["mixer"].update(dim=300),
    "a routed feed-forward": lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    "a width in words": lambda c: c.update(width="64"),
}


@pytest.mark.parametrize("what", sorted(BAD))
def test_refusals_name_the_key(what):
    raw = copy.deepcopy(CONFIGS["A"])
    BAD[what](raw)
    with pytest.raises(ConfigError):
        config_from_normalised(raw).validate()


def test_cache_layout_of_shared_and_windowed_entries():
    """Attention layers have pages; an entry that two layers read keeps what the longer window and the longer start need;
    recurrences have a state and no pages."""
    from sandyrt_b200.models.model import build_model

    specs = build_model(config_from_normalised(CONFIGS["A"])).cache_specs()
    assert [s["kind"] for s in specs] == ["paged", "state", "state", "state"]
    assert (specs[0]["window"], specs[0]["keep_first"], specs[0]["head_dim"], specs[0]["n_kv_heads"]) == (40, 5, 32, 2)
    assert specs[1]["shape"] == [2 * 16 * 24] and specs[3]["shape"] == [3 * 24 * 8]
    specs = build_model(config_from_normalised(CONFIGS["B"])).cache_specs()
    assert (specs[1]["window"], specs[1]["keep_first"]) == (0, 0)           # one of the two readers looks back over everything
    assert (specs[3]["window"], specs[3]["keep_first"]) == (1, 1)
    assert all(s["kind"] == "state" for s in build_model(config_from_normalised(CONFIGS["D"])).cache_specs())


def test_pages_behind_a_window_go_back_but_for_the_kept_ones():
    """Pages of 4, a window of 10, 6 kept positions (two pages): blocks 2, 3, .. are given back as the window passes them,
    blocks 0 and 1 never; everything at the end."""
    from sandyrt_b200.cache.pages import FREED, BlockAllocator, CacheLayout
    from sandyrt_b200.parts.base import PagedKVSpec

    layout = CacheLayout.from_specs([PagedKVSpec(1, 16, window=10, keep_first=6), PagedKVSpec(1, 16, window=10)], 4)
    assert len(layout.groups) == 2                                         # the needs differ
    al = BlockAllocator(layout, [20, 20], 2)
    al.admit("r")
    for n in (3, 9, 10, 17, 18, 19, 40, 61):
        al.reserve("r", n)
        al.commit("r", n)
        al.check()
        first = max(0, n - 10 + 1) // 4
        kept, plain_window = al.block_list("r", 0), al.block_list("r", 1)
        for b in range(len(kept)):
            assert (kept[b] == FREED) == (2 <= b < first), (n, b)
            assert (plain_window[b] == FREED) == (b < first), (n, b)
    assert al.free_pages(0) == 20 - 2 - sum(1 for b in al.block_list("r", 0)[2:] if b != FREED)
    al.release("r")
    al.check()
    assert al.free_pages(0) == 20 and al.free_pages(1) == 20


def test_a_scheduler_counts_the_kept_pages():
    """A prompt of 200 through a window of 16 that keeps 32 positions, pages of 16, portions of 16: the window and the
    portion take three pages, the kept positions two more; with those five the request runs to its end."""
    from sandyrt_b200.cache.pages import BlockAllocator, CacheLayout
    from sandyrt_b200.engine.scheduler import Request, RequestRefused, Scheduler
    from sandyrt_b200.parts.base import PagedKVSpec

    def sched(pages):
        alloc = BlockAllocator(CacheLayout.from_specs([PagedKVSpec(1, 16, window=16, keep_first=32)], 16), [pages], 2)
        return Scheduler(alloc, max_step_tokens=32, prefill_chunk=16, max_live=2), alloc

    with pytest.raises(RequestRefused):
        sched(4)[0].add(Request("r", list(range(200)), 9))
    s, alloc = sched(5)
    s.add(Request("r", list(range(200)), 9))
    steps = 0
    while s.has_work():
        plan = s.plan()
        assert plan.portions
        s.complete(plan, {p.request.rid: 7 for p in plan.portions if p.samples})
        alloc.check()
        steps += 1
        assert steps < 100
    assert alloc.free_pages(0) == 5


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_mask_edges():
    seen = plain.visible(12, 4, 2)
    assert seen[9].nonzero().flatten().tolist() == [0, 1, 6, 7, 8, 9]
    assert seen[4].nonzero().flatten().tolist() == [0, 1, 2, 3, 4]
    assert seen[1].nonzero().flatten().tolist() == [0, 1]
    assert plain.visible(6, 0, 0).equal(torch.ones(6, 6, dtype=torch.bool).tril())
    assert plain.visible(5, 1, 3)[4].nonzero().flatten().tolist() == [0, 1, 2, 4]


def test_plain_rotation_pairs_neighbours_and_leaves_the_rest():
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    y = plain.rotate(x, torch.arange(5), 4, 100.0)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    a = 3 * 100.0 ** (-2.0 / 4)
    assert math.isclose(float(y[3, 1, 2]), float(x[3, 1, 2] * math.cos(a) - x[3, 1, 3] * math.sin(a)), rel_tol=1e-12)
    assert math.isclose(float(y[3, 1, 3]), float(x[3, 1, 3] * math.cos(a) + x[3, 1, 2] * math.sin(a)), rel_tol=1e-12)


def test_plain_softmax_with_one():
    s = torch.tensor([[0.5, -1.0, float("-inf")], [-300.0, -400.0, float("-inf")]], dtype=torch.float64)
    p = plain.softmax_with_one(s)
    den = 1 + math.exp(0.5) + math.exp(-1.0)
    assert torch.allclose(p[0], torch.tensor([math.exp(0.5) / den, math.exp(-1.0) / den, 0.0], dtype=torch.float64))
    assert p[1].sum() < 1e-100


def test_plain_recurrences_carry_on():
    """Token by token from a state equals the whole sequence; a channel whose factor is zero forgets everything before."""
    torch.manual_seed(0)
    q, k, la = torch.randn(9, 5).double(), torch.randn(9, 5).double(), -torch.rand(9, 5).double()
    v = torch.randn(9, 3).double()
    whole, _ = plain.gla_rule(q, k, v, la)
    a, S = plain.gla_rule(q[:4], k[:4], v[:4], la[:4])
    b, _ = plain.gla_rule(q[4:], k[4:], v[4:], la[4:], S)
    assert torch.allclose(torch.cat([a, b]), whole)
    la[6] = -1e9
    assert torch.allclose(plain.gla_rule(q, k, v, la)[0][6], (k[6] @ q[6]) * v[6])
    li, lf = torch.randn(9).double(), -torch.rand(9).double()
    whole, _ = plain.mlstm_rule(q, k, v, li, lf)
    a, st = plain.mlstm_rule(q[:2], k[:2], v[:2], li[:2], lf[:2])
    assert torch.allclose(torch.cat([a, plain.mlstm_rule(q[2:], k[2:], v[2:], li[2:], lf[2:], st)[0]]), whole)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plain_is_causal(name):
    cfg = CONFIGS[name]
    w = make_weights(cfg, seed=1)
    ids = list(range(3, 40))
    full = plain.forward(cfg, w, ids)
    assert torch.allclose(plain.forward(cfg, w, ids[:20]), full[:20], atol=1e-9)
    other = list(ids)
    other[30] = 50
    again = plain.forward(cfg, w, other)
    assert torch.allclose(again[:30], full[:30], atol=1e-9) and not torch.allclose(again[30], full[30], atol=1e-3)
