"""Migelix without a GPU: the configuration and its checks, the model description (parts, run order, layers on another's
tensors, tensor names), the cache entries, and properties of the plain implementation that the GPU tests lean on."""
import copy
import math

import pytest
import torch

import plain_migelix as plain
from migelix_models import CONFIGS, _config, attention, delta, heads_of, layer, make_weights, parallel, tensor_shapes, without_ranks, wkv

from sandyrt_b200.config.base import ConfigError, config_from_normalised
from sandyrt_b200.config.migelix import MigelixConfig


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_description_names_every_tensor_with_its_shape(name):
    from sandyrt_b200.models.model import build_model

    cfg = config_from_normalised(CONFIGS[name])
    assert isinstance(cfg, MigelixConfig) and cfg.vocab_size == CONFIGS[name]["vocab"]
    cfg.validate()
    got = {k: list(v.shape) for k, v in build_model(cfg).tensor_requests().items()}
    assert got == tensor_shapes(CONFIGS[name])
    # the ranks are the weight file's where the configuration is silent
    got = {k: list(v.shape) for k, v in build_model(config_from_normalised(without_ranks(CONFIGS[name]))).tensor_requests().items()}
    for k, v in tensor_shapes(CONFIGS[name]).items():
        last = k.split(".")[-1]
        assert got[k] == ([-1, v[1]] if last in ("a1", "g1", "w1") else [v[0], -1] if last in ("a2", "g2", "w2") else v)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_run_order_and_cache_entries(name):
    """Every layer has a cache entry of its own; one with weights_of runs another layer's parts."""
    from sandyrt_b200.models.model import describe

    raw = CONFIGS[name]
    spec = describe(config_from_normalised(raw))
    own = [i for i, l in enumerate(raw["layers"]) if l.get("weights_of") is None]
    assert len(spec.layers) == len(own)
    assert [c.layer for c in spec.schedule] == [own.index(plain.tensors_of(raw, i)) for i in range(len(raw["layers"]))]
    assert [c.cache for c in spec.schedule] == list(range(len(raw["layers"]))) and all(c.write_cache for c in spec.schedule)
    kinds = {"attention": "windowed_attention", "parallel": "attention_beside_channel_delta", "wkv": "time_mixing"}
    for i, s in zip(own, spec.layers):
        l = raw["layers"][i]
        assert s.block == "pre_norm" and sorted(s.norms) == (["feed_forward", "mixer"] if l["mlp"] else ["mixer"])
        assert s.mixer.kind == kinds[l["type"]] and s.feed_forward.kind == ("gated_mlp" if l["mlp"] else "none")
        assert all(n.params["gain_offset"] == 1.0 and n.params["eps"] == raw["norm"]["eps"] for n in s.norms.values())
    assert spec.final_norm.params["gain_offset"] == 1.0 and spec.head.params["tied"] is True and spec.max_positions is None
    assert spec.head.params.get("logit_softcap") == raw.get("logit_softcap")


def test_config_round_trip_and_constants_reach_the_parts():
    from sandyrt_b200.models.model import describe

    raw = CONFIGS["A"]
    cfg = MigelixConfig.from_dict(raw)
    assert MigelixConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.to_dict()["layers"] == raw["layers"] and cfg.to_dict()["logit_softcap"] == 20.0
    spec = describe(cfg)
    m = spec.layers[1].mixer.params
    assert (m["n_heads"], m["n_kv_heads"], m["qk_dim"], m["v_dim"], m["window"], m["softcap"]) == (4, 2, 16, 16, 24, 6.0)
    assert m["values_are_keys"] and m["rot_interleaved"] and m["out_gate"] and "bias" not in m and "sink" not in m and "rot_yarn" not in m
    p = spec.layers[2].mixer.params
    assert (p["left_scale"], p["right_scale"], p["left.rot_dims"], p["left.rot_base"], p["left.window"]) == (0.7, 1.4, 12, 50.0, 17)
    assert p["left.rot_yarn"] == {"factor": 4.0, "original": 30.0, "fast": 8.0, "slow": 1.0} and p["left.sink"] and p["left.bias"]
    assert [p["right." + k] for k in ("n_heads", "n_qk_heads", "qk_dim", "v_dim", "conv_taps", "rank", "gate_rank")] == [4, 2, 16, 24, 4, 6, 5]
    assert spec.layers[2].mixer.tensors["right.decay_in"] == "l2.mix.right.a1" and spec.layers[0].mixer.tensors["mu_w"] == "l0.mix.mu.w"


def test_optional_keys_have_their_defaults():
    raw = _config(31, 16, [layer(attention(2, 2, 8), None), layer(parallel(heads_of(2, 2, 8), delta(1, 1, 4, 4)), None)], cap=None)
    for m in (raw["layers"][0]["mixer"], raw["layers"][1]["mixer"]["left"], raw["layers"][1]["mixer"]["right"]):
        del m["kv_heads"]
    raw["layers"][0]["mixer"].update(mask=None, rot=None, softcap=None)
    raw["layers"][0]["weights_of"] = None
    cfg = config_from_normalised(raw)
    cfg.validate()
    assert cfg.logit_softcap == 0.0 and cfg.to_dict()["layers"][1]["mixer"]["right"]["kv_heads"] == 1
    assert cfg.to_dict()["layers"][0]["mixer"]["kv_heads"] == 2 and "softcap" not in cfg.to_dict()["layers"][0]["mixer"]


def test_a_layer_may_use_the_tensors_of_one_that_uses_anothers():
    from sandyrt_b200.models.model import describe

    raw = _config(31, 16, [layer(wkv(1, 8), None), layer(attention(2, 1, 8), 12)], reuse=(0, 1))
    raw["layers"].append(dict(copy.deepcopy(raw["layers"][0]), weights_of=2))
    cfg = config_from_normalised(raw)
    cfg.validate()
    assert [c.layer for c in describe(cfg).schedule] == [0, 1, 0, 1, 0]


BAD = {
    "no width": lambda c: c.pop("width"),
    "no layers": lambda c: c.update(layers=[]),
    "an unknown layer type": lambda c: c["layers"][0].update(type="lstm"),
    "heads that do not divide": lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
    "query heads of the delta rule that do not divide": lambda c: c["layers"][2]["mixer"]["right"].update(kv_heads=3),
    "an odd number of rotated entries": lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    "more rotated entries than a head has": lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18),
    "values of another size than keys": lambda c: c["layers"][1]["mixer"].update(vdim=8),
    "a negative window": lambda c: c["layers"][1]["mixer"]["mask"].update(size=-1),
    "a negative cap": lambda c: c["layers"][1]["mixer"].update(softcap=-1.0),
    "a negative cap of the logits": lambda c: c.update(logit_softcap=-1.0),
    "no scale beside the delta rule": lambda c: c["layers"][2]["mixer"].pop("left_scale"),
    "a rescaling without its factor": lambda c: c["layers"][2]["mixer"]["left"]["rot"]["scaling"].pop("factor"),
    "a rescaling by zero": lambda c: c["layers"][2]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0),
    "too many taps": lambda c: c["layers"][2]["mixer"]["right"].update(conv=9),
    "a state beyond the kernels": lambda c: c["layers"][0]["mixer"].update(dim=300),
    "tensors of a layer that is not there": lambda c: c["layers"][3].update(weights_of=17),
    "tensors in a circle": lambda c: c["layers"][2].update(weights_of=3),
    "tensors of a layer of other sizes": lambda c: c["layers"][3]["mixer"]["right"].update(vdim=8),
    "tensors of a layer of other constants": lambda c: c["layers"][3]["mixer"].update(left_scale=0.5),
    "a routed feed-forward": lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    "a width in words": lambda c: c.update(width="64"),
}


@pytest.mark.parametrize("what", sorted(BAD))
def test_refusals_name_the_key(what):
    raw = copy.deepcopy(CONFIGS["A"])
    BAD[what](raw)
    with pytest.raises(ConfigError):
        config_from_normalised(raw).validate()


def test_cache_entries_hold_pages_states_or_both():
    from sandyrt_b200.models.model import build_model

    specs = build_model(config_from_normalised(CONFIGS["A"])).cache_specs()
    assert [s["kind"] for s in specs] == ["state", "paged", "paged_state", "paged_state", "state", "paged"]
    assert specs[0]["shape"] == [64 + 3 * 16 * 16] and (specs[1]["window"], specs[1]["head_dim"], specs[1]["n_kv_heads"]) == (24, 16, 2)
    assert (specs[2]["window"], specs[2]["head_dim"]) == (17, 32)
    assert specs[2]["shape"] == [4 * 16 * 24 + 3 * (2 * 2 * 16 + 4 * 24)]
    assert all(s["kind"] == "state" for s in build_model(config_from_normalised(CONFIGS["D"])).cache_specs())


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_mask_edges():
    seen = plain.visible(12, 4)
    assert seen[9].nonzero().flatten().tolist() == [6, 7, 8, 9] and seen[1].nonzero().flatten().tolist() == [0, 1]
    assert plain.visible(6, 0).equal(torch.ones(6, 6, dtype=torch.bool).tril()) and plain.visible(5, 1).equal(torch.eye(5, dtype=torch.bool))


def test_plain_rotation_pairs_neighbours_and_leaves_the_rest():
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    y = plain.rotate(x, torch.arange(5), 4, 100.0, None)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    a = 3 * 100.0 ** (-2.0 / 4)
    assert math.isclose(float(y[3, 1, 2]), float(x[3, 1, 2] * math.cos(a) - x[3, 1, 3] * math.sin(a)), rel_tol=1e-12)
    assert math.isclose(float(y[3, 1, 3]), float(x[3, 1, 3] * math.cos(a) + x[3, 1, 2] * math.sin(a)), rel_tol=1e-12)


def test_plain_yarn_keeps_fast_pairs_and_slows_slow_ones():
    s = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    f, m = plain.yarn(64, 10000.0, s)
    base, one = plain.yarn(64, 10000.0, None)
    assert one == 1.0 and math.isclose(m, 0.1 * math.log(4.0) + 1.0)
    turns = [4096 * b / (2 * math.pi) for b in base]
    lo = next(i for i, t in enumerate(turns) if t < 32.0)
    hi = next(i for i, t in enumerate(turns) if t < 1.0)
    assert f[:lo - 1] == base[:lo - 1] and lo > 2 and hi < 30
    # the pair's index is compared with entry numbers of the whole rotated part, twice as many as pairs
    ratios = [a / b for a, b in zip(f, base)]
    assert ratios == sorted(ratios, reverse=True) and all(0.25 <= r <= 1.0 for r in ratios)
    x = torch.ones(1, 1, 2, dtype=torch.float64)
    assert math.isclose(float(plain.rotate(x, torch.zeros(1), 2, 100.0, s)[0, 0, 0]), m, rel_tol=1e-12)


def test_plain_attention_with_a_sink_and_a_cap():
    q, k = torch.tensor([[[2.0]]]).double(), torch.tensor([[[3.0]]]).double()
    v, seen = torch.tensor([[[5.0]]]).double(), torch.ones(1, 1, dtype=torch.bool)
    assert float(plain.attention_heads(q, k, v, 0.5, seen)[0, 0, 0]) == 5.0
    sink = torch.tensor([1.0]).double()
    want = 5.0 * math.exp(3.0) / (math.exp(3.0) + math.exp(1.0))
    assert math.isclose(float(plain.attention_heads(q, k, v, 0.5, seen, 0.0, sink)[0, 0, 0]), want, rel_tol=1e-12)
    capped = 2.0 * math.tanh(1.5)
    want = 5.0 * math.exp(capped) / (math.exp(capped) + math.exp(1.0))
    assert math.isclose(float(plain.attention_heads(q, k, v, 0.5, seen, 2.0, sink)[0, 0, 0]), want, rel_tol=1e-12)


def test_plain_recurrences_carry_on():
    """Token by token from a state equals the whole sequence; the delta rule reads back what it has just written when nothing
    fades and the step is whole; the bonus reaches the current token only."""
    torch.manual_seed(0)
    q, k, la = torch.randn(9, 5).double(), plain.unit(torch.randn(9, 5).double()), -torch.rand(9, 5).double()
    v, beta, u = torch.randn(9, 3).double(), torch.rand(9).double(), torch.randn(5).double()
    for rule, args in ((plain.delta_rule, lambda a, b: (q[a:b], k[a:b], v[a:b], beta[a:b], la[a:b])),
                       (plain.wkv_rule, lambda a, b: (q[a:b], k[a:b], v[a:b], u, la[a:b]))):
        whole, _ = rule(*args(0, 9))
        head, S = rule(*args(0, 4))
        assert torch.allclose(torch.cat([head, rule(*args(4, 9), S)[0]]), whole)
    ones, zero = torch.ones(9).double(), torch.zeros(9, 5).double()
    _, S = plain.delta_rule(q, k, v, ones, zero)
    assert torch.allclose(S.t() @ k[8], v[8], atol=1e-5)
    assert torch.allclose(plain.wkv_rule(q, k, v, u, la)[0][0], (q[0] * u) @ k[0] * v[0])


def test_plain_short_convolution():
    x, taps = torch.arange(1.0, 7.0).view(6, 1), torch.tensor([[100.0, 10.0, 1.0]])
    assert plain.short_conv(x, taps)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0, 456.0]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plain_is_causal(name):
    cfg = CONFIGS[name]
    w = make_weights(cfg, seed=1)
    ids = list(range(3, 40))
    full = plain.forward(cfg, w, ids)
    assert torch.allclose(plain.forward(cfg, w, ids[:20]), full[:20], atol=1e-9)
    other = list(ids)
    other[30] = 50
    changed = plain.forward(cfg, w, other)
    assert torch.allclose(changed[:30], full[:30], atol=1e-9) and not torch.allclose(changed[30], full[30], atol=1e-3)
