"""Migelix configurations drawn at random, each through the engine whole, as a prompt with single tokens behind it and in
portions, in both compute types, against the plain implementation (tests/plain_migelix.py).

The sizes divide by nothing in particular: widths of 44 to 136 (some no multiple of 8), head sizes of 2 to 128, fewer query/key
heads than heads, windows of 1 to 60 tokens or none, rotations of all or a part of a head with and without rescaling, 1 to 8 taps,
ranks of 1 to 20, layers on another's tensors.  Bounds as in test_migelix_gpu.py."""
import numpy as np
import pytest
import torch

import plain_migelix as plain
from migelix_models import _config, attention, delta, heads_of, layer, make_weights, parallel, rel_error, wkv, write_model

pytestmark = pytest.mark.gpu


def draw(seed: int) -> dict:
    r = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(r.integers(0, len(xs)))]

    def attending():
        kv, dim = int(pick(1, 2, 3)), int(pick(2, 6, 8, 16, 24, 40, 64, 64, 80, 128))
        rot = 2 * int(r.integers(0, dim // 2 + 1))
        yarn = (float(pick(2.0, 4.0, 9.0)), float(pick(20, 64, 300)), float(pick(4.0, 32.0)), float(pick(0.5, 1.0, 2.0))) if r.random() < 0.6 else None
        return dict(heads=kv * int(pick(1, 2, 5)), kv_heads=kv, dim=dim, size=int(r.integers(1, 61)) if r.random() < 0.8 else 0, rot=rot or None,
                    base=float(pick(30.0, 1e3, 5e5)), yarn=yarn, scale=float(pick(0.1, 0.3, 0.6)))

    layers = []
    for i in range(int(r.integers(1, 5))):
        ff = int(pick(8, 20, 44, 64)) if r.random() < 0.6 else None
        kind = pick("attention", "parallel", "parallel", "wkv")
        if kind == "attention":
            a = attending()
            a.pop("yarn")
            mixer = attention(**a, softcap=float(pick(1.5, 5.0, 30.0)))
        elif kind == "parallel":
            G = int(pick(1, 2, 3))
            mixer = parallel(heads_of(**attending()), delta(G * int(pick(1, 2, 3)), G, int(pick(2, 7, 16, 24, 64, 72)), int(pick(3, 8, 12, 30, 64, 72)),
                             conv=int(r.integers(1, 9)), rank=int(r.integers(1, 21)), gate_rank=int(r.integers(1, 21))),
                             float(pick(1.0, 0.4, -1.3)), float(pick(1.0, 0.8, 1.9)))
        else:
            mixer = wkv(int(pick(1, 2, 3, 5)), int(pick(2, 7, 16, 24, 40, 64, 72)), rank=int(r.integers(1, 21)))
        layers.append(layer(mixer, ff))
    reuse = [int(r.integers(0, len(layers))) for _ in range(int(r.integers(0, 3)))]
    return _config(int(r.integers(40, 150)), int(pick(44, 48, 66, 72, 90, 100, 128, 136)), layers, eps=float(pick(1e-5, 1e-6, 1e-3)),
                   cap=pick(None, 5.0, 25.0), reuse=reuse)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(20))
def test_a_configuration_drawn_at_random(tmp_path, seed, dtype):
    from sandyrt_b200.engine.step import Engine, StepEntry
    from sandyrt_b200.models.model import load_model

    cfg = draw(seed)
    ids = np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], size=90).tolist()
    w = make_weights(cfg, seed=seed)
    path = write_model(cfg, w, str(tmp_path / "m"))
    want = plain.forward(cfg, w, ids).numpy()
    run = plain.forward(cfg, w, ids, dtype=torch.float32) if dtype == "float32" else plain.forward_rounded(cfg, w, ids)
    bound = max(2e-4 if dtype == "float32" else 2e-2, 3 * rel_error(run.numpy(), want))
    eng = Engine(load_model(path, device="cuda:0", dtype=getattr(torch, dtype)), max_tokens=128, page_size=8, max_requests=2)
    eng.cache.device_caches.poison()
    for cuts in ([90], [61] + [1] * 29, [2, 9, 1, 30, 3, 45]):
        rows, pos = [], 0
        for n in cuts:
            rows.append(eng.step([StepEntry("r", ids[pos:pos + n], list(range(n)))]).cpu().numpy().copy())
            pos += n
        eng.check_status()
        eng.release("r")
        e = rel_error(np.concatenate(rows), want)
        assert e < bound, f"seed {seed}, cuts {cuts[:4]}: relative error {e:.3e} (bound {bound:.1e}); {cfg}"
