"""Pugalix configurations drawn at random, each through the engine whole, as a prompt with single tokens behind it and in
portions, in both compute types, against the plain implementation (tests/plain_pugalix.py).

The sizes divide by nothing in particular: widths of 44 to 136 (some no multiple of 8), head sizes of 2 to 80 with query
and value sizes apart, windows of 1 to 60 tokens that keep 0 to 40, readers of earlier layers with windows of their own,
decays of rank 1 to 20 and tau of 0.5 to 30, gate caps of 2 to 25.  Bounds as in test_pugalix_gpu.py."""
import numpy as np
import pytest
import torch

import plain_pugalix as plain
from pugalix_models import _config, attention, gla, layer, make_weights, mlstm, rel_error, write_model

pytestmark = pytest.mark.gpu


def draw(seed: int) -> dict:
    r = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(r.integers(0, len(xs)))]
    layers, writers = [], []
    for i in range(int(r.integers(1, 7))):
        ff = int(pick(8, 20, 44, 64)) if r.random() < 0.6 else None
        kind = pick("attention", "attention", "gla", "mlstm")
        if kind == "attention":
            window = dict(size=int(r.integers(1, 61)), keep=int(pick(0, 1, 3, 8, 17, 40))) if r.random() < 0.8 else {}
            if writers and r.random() < 0.5:
                src = int(pick(*writers))
                m = layers[src]["mixer"]
                mixer = attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], scale=float(pick(0.1, 0.3, 0.6)), kv_from=src, **window)
                if "rot" in m:
                    mixer["mixer"]["rot"] = dict(m["rot"])
            else:
                kv, dim = int(pick(1, 2, 3)), int(pick(2, 6, 8, 16, 24, 40, 64, 64, 80))
                rot = 2 * int(r.integers(0, dim // 2 + 1))
                mixer = attention(kv * int(pick(1, 2, 5)), kv, dim, int(pick(3, 8, 16, 20, 48, 64, 64)), rot=rot or None,
                                  base=float(pick(30.0, 1e3, 5e5)), scale=float(pick(0.1, 0.3, 0.6)), **window)
                writers.append(i)
        elif kind == "gla":
            mixer = gla(int(pick(1, 2, 3, 5)), int(pick(2, 7, 16, 24, 40, 64, 72)), int(pick(3, 8, 12, 30, 64, 72)), tau=float(pick(0.5, 1.0, 5.0, 16.0, 30.0)),
                        rank=int(r.integers(1, 21)))
        else:
            mixer = mlstm(int(pick(1, 2, 3, 5)), int(pick(2, 7, 16, 24, 40, 64, 72)), int(pick(3, 8, 12, 30, 64, 72)), cap=float(pick(2.0, 8.0, 15.0, 25.0)))
        layers.append(layer(mixer, ff))
    return _config(int(r.integers(40, 150)), int(pick(44, 48, 66, 72, 90, 100, 128, 136)), layers, scale=float(pick(1.0, 0.3, 4.0, 11.3)),
                   eps=float(pick(1e-5, 1e-6)))


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
