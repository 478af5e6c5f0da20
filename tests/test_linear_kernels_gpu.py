"""Kernels of the windowed attention and of the gated linear attention, each alone against a plain float64 formula: kept
first keys behind a window and a gate by element in every attention kernel that has a form for them, rotation of
neighbouring pairs, the recurrence with a decay per key channel token by token and in chunks."""
import math

import pytest
import torch

from test_kernels_gpu import ATT_TOL, DEV, _paged_case

pytestmark = pytest.mark.gpu


# ---- attention ---------------------------------------------------------------------------------------------------
def _want(case, H, Hkv, scale, window, keep, sink, gate, dim):
    """Query at pos sees keys of the last `window` positions and the first `keep`; a sink of one in the denominator; entry
    i < dim of head h's output times sigmoid(gate[t, h * dim + i])."""
    outs, t = [], 0
    for s, (before, n) in enumerate(case["seqs"]):
        k, v, q = case["dense_k"][s].double(), case["dense_v"][s].double(), case["qs"][s].double()
        for i in range(n):
            pos = before + i
            j = torch.arange(pos + 1)
            seen = (j > pos - window) | (j < keep) if window else j >= 0
            row = []
            for h in range(H):
                kh = h // (H // Hkv)
                p = torch.exp((k[:pos + 1, kh][seen] @ q[i, h]) * scale)
                o = (p @ v[:pos + 1, kh][seen]) / (p.sum() + (1.0 if sink else 0.0))
                if gate is not None:
                    o = o.clone()
                    o[:dim] *= torch.sigmoid(gate[t, h * dim:(h + 1) * dim])
                row.append(o)
            outs.append(torch.cat(row))
            t += 1
    return torch.stack(outs)


def _gate(case, H, dim, seed):
    """A column range of a wider matrix, so that its pitch is not its width."""
    T, dt = case["q"].shape[0], case["q"].dtype
    wide = torch.randn(T, H * dim + 24, generator=torch.Generator().manual_seed(seed)).mul(2).to(dt).to(DEV)
    return wide[:, 8:8 + H * dim]


SHAPES = [(4, 2, 16, 16, 40, 5), (5, 5, 48, 8, 64, 64), (6, 2, 64, 16, 1, 1), (12, 12, 64, 16, 100, 19), (4, 1, 128, 32, 33, 3), (3, 1, 80, 4, 10, 30)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Hkv,D,page_size,window,keep", SHAPES + [(2, 1, 144, 16, 20, 7)])
def test_general_kernel(dtype, H, Hkv, D, page_size, window, keep):
    from sandyrt_b200.csrc import ops

    seqs = [(0, 33), (window + keep - 1, 4), (17, 24), (0, 1), (230, 1), (keep, 2)]
    case = _paged_case(dtype, H, Hkv, D, page_size, seqs, seed=D + H)
    dim = D - 5
    gate = _gate(case, H, dim, seed=D)
    scale = 0.7 / math.sqrt(D)
    out = torch.full_like(case["q"], float("nan"))
    args = (case["q"], case["kc"], case["vc"], case["table"], case["tok_seq"], case["tok_pos"], out)
    zero = torch.zeros(H, device=DEV)
    ops.paged_attention(*args, n_heads=H, scale=scale, window=window, keep_first=keep, sink=zero, elem_gate=gate)
    ops.check_kernel_status(DEV)
    assert (out.double().cpu() - _want(case, H, Hkv, scale, window, keep, True, gate.double().cpu(), dim)).abs().max().item() < ATT_TOL[dtype] * 1.5
    # without kept keys and gate: the plain window, bit for bit
    plain_out = torch.empty_like(out)
    ops.paged_attention(*args[:-1], plain_out, n_heads=H, scale=scale, window=window)
    ops.paged_attention(*args, n_heads=H, scale=scale, window=window, keep_first=0)
    assert torch.equal(out, plain_out)


@pytest.mark.parametrize("H,Hkv,D,page_size,window,keep", SHAPES)
@pytest.mark.parametrize("splits", [1, 3, 8])
@pytest.mark.parametrize("kind", ["rows", "mma"])
def test_decode_kernels(kind, H, Hkv, D, page_size, window, keep, splits):
    """Single tokens whose windows begin before, at and behind the kept keys' end and at page borders."""
    from sandyrt_b200.csrc import ops

    if kind == "mma" and D != 64:
        pytest.skip("heads of 64")
    seqs = [(699, 1), (0, 1), (63, 1), (300, 1)] + [(max(0, window + keep + d), 1) for d in (-2, -1, 0, 1, 2)] + [(window - 1, 1), (window, 1)]
    case = _paged_case(torch.bfloat16, H, Hkv, D, page_size, seqs, seed=D + splits)
    dim = D - 3
    gate = _gate(case, H, dim, seed=splits)
    scale = 1.0 / math.sqrt(D)
    out = torch.full_like(case["q"], float("nan"))
    args = (case["q"], case["kc"], case["vc"], case["table"], case["tok_seq"], case["tok_pos"], out)
    kw = dict(n_heads=H, scale=scale, window=window, keep_first=keep, sink=torch.zeros(H, device=DEV), elem_gate=gate)
    if kind == "mma":
        ops.decode_attention(*args, num_splits=splits, mma=True, **kw)
    else:
        ops.decode_attention_shared(*args, splits=splits, **kw)
    ops.check_kernel_status(DEV)
    want = _want(case, H, Hkv, scale, window, keep, True, gate.double().cpu(), dim)
    assert (out.double().cpu() - want).abs().max().item() < ATT_TOL[torch.bfloat16] * 1.5


@pytest.mark.parametrize("H,Hkv,D,page_size,window,keep,tc", [(s + (False,)) for s in SHAPES] +
                         [(4, 2, 64, 16, 40, 5, True), (12, 12, 64, 16, 129, 130, True), (3, 3, 64, 8, 300, 7, True), (2, 2, 64, 16, 1, 1, True)])
def test_prompt_kernels(H, Hkv, D, page_size, window, keep, tc):
    """Portions whose rows' windows leave whole key tiles between the kept keys and themselves, beside single tokens and a
    first portion whose rows still see everything."""
    from sandyrt_b200.csrc import ops

    seqs = [(0, 150), (520, 70), (17, 70), (0, 1), (640, 3), (301, 1)]
    case = _paged_case(torch.bfloat16, H, Hkv, D, page_size, seqs, seed=D + H, runs=(0, 1))
    dim = D - 2
    gate = _gate(case, H, dim, seed=H)
    scale = 1.0 / math.sqrt(D)
    q_start = torch.tensor([0] + list(torch.tensor([n for _, n in seqs]).cumsum(0)), dtype=torch.int32, device=DEV)
    kv_before = torch.tensor([b for b, _ in seqs], dtype=torch.int32, device=DEV)
    out = torch.full_like(case["q"], float("nan"))
    ops.prefill_attention(case["q"], case["kc"], case["vc"], case["table"], q_start, kv_before, out, n_heads=H, max_q_len=150, scale=scale,
                          tc=tc, window=window, keep_first=keep, sink=torch.zeros(H, device=DEV), elem_gate=gate)
    ops.check_kernel_status(DEV)
    want = _want(case, H, Hkv, scale, window, keep, True, gate.double().cpu(), dim)
    assert (out.double().cpu() - want).abs().max().item() < ATT_TOL[torch.bfloat16] * 1.5


@pytest.mark.parametrize("tc", [False, True])
def test_pages_between_the_kept_keys_and_the_window_may_be_gone(tc):
    """The block table names no page for the blocks that the window has left behind and the kept keys do not need: no
    kernel reads them or reports them, and the result is the same."""
    from sandyrt_b200.csrc import ops

    H, D, page, window, keep = 4, 64, 16, 50, 20
    seqs = [(400, 40), (300, 1)]
    case = _paged_case(torch.bfloat16, H, H, D, page, seqs, seed=3)
    table = case["table"].clone()
    for s, (before, n) in enumerate(seqs):
        first = (before + 1 - window) // page
        table[s, 2:first] = -1                                   # the kept keys take blocks 0 and 1
    q_start = torch.tensor([0, 40, 41], dtype=torch.int32, device=DEV)
    kv_before = torch.tensor([400, 300], dtype=torch.int32, device=DEV)
    out = torch.full_like(case["q"], float("nan"))
    ops.prefill_attention(case["q"], case["kc"], case["vc"], table, q_start, kv_before, out, n_heads=H, max_q_len=40, scale=0.125, tc=tc,
                          window=window, keep_first=keep)
    ops.check_kernel_status(DEV)
    want = _want(case, H, H, 0.125, window, keep, False, None, D)
    assert (out.double().cpu() - want).abs().max().item() < ATT_TOL[torch.bfloat16]
    one = [x[40:41] if x.dim() == 2 else x[40:41].contiguous() for x in (case["q"], case["tok_seq"], case["tok_pos"])]
    for kind in ("rows", "mma", "general"):
        got = torch.full_like(one[0], float("nan"))
        args = (one[0], case["kc"], case["vc"], table, one[1], one[2], got)
        kw = dict(n_heads=H, scale=0.125, window=window, keep_first=keep)
        if kind == "rows":
            ops.decode_attention_shared(*args, splits=2, **kw)
        elif kind == "mma":
            ops.decode_attention(*args, num_splits=2, mma=True, **kw)
        else:
            ops.paged_attention(*args, **kw)
        ops.check_kernel_status(DEV)
        assert (got.double().cpu() - want[40:41]).abs().max().item() < ATT_TOL[torch.bfloat16], kind


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Hkv,d,e,rot,interleaved", [(4, 2, 16, 24, 8, True), (3, 1, 20, 12, 20, True), (2, 2, 64, 64, 32, False), (5, 5, 12, 12, 2, True)])
def test_rotation_of_neighbours_and_halves(dtype, H, Hkv, d, e, rot, interleaved):
    """Queries and keys turned and padded, values as they are; with write_cache off the pages stay untouched."""
    from sandyrt_b200.csrc import ops

    T, page, D = 23, 8, -(-max(d, e) // 16) * 16
    g = torch.Generator().manual_seed(d)
    proj = torch.randn(T, H * d + Hkv * (d + e) + 5, generator=g).to(dtype).to(DEV)
    pos = torch.arange(11, 11 + T, dtype=torch.int32, device=DEV)
    arena = torch.full((8, 2, Hkv, page, D), 7.0, dtype=dtype, device=DEV)
    kc, vc = arena[:, 0], arena[:, 1]
    table = torch.tensor([[5, 3, 1, 0, 2, 4]], dtype=torch.int32, device=DEV)
    seq = torch.zeros(T, dtype=torch.int32, device=DEV)
    freq = torch.tensor([30.0 ** (-2 * i / rot) for i in range(rot // 2)], device=DEV)
    q = torch.full((T, H * D), float("nan"), dtype=dtype, device=DEV)
    ops.attention_prepare(proj, kc, vc, table, seq, pos, q, n_heads=H, qk_dim=d, v_dim=e, freq=freq, interleaved=interleaved, write_cache=False)
    assert (arena == 7.0).all()
    ops.attention_prepare(proj, kc, vc, table, seq, pos, q, n_heads=H, qk_dim=d, v_dim=e, freq=freq, interleaved=interleaved)
    ops.check_kernel_status(DEV)

    def turn(x):
        x = x.double().cpu().clone()
        y = x.clone()
        for i in range(rot // 2):
            a = torch.arange(11, 11 + T).double() * float(freq[i])
            i0, i1 = (2 * i, 2 * i + 1) if interleaved else (i, i + rot // 2)
            c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
            y[:, :, i0] = x[:, :, i0] * c - x[:, :, i1] * s
            y[:, :, i1] = x[:, :, i1] * c + x[:, :, i0] * s
        return y

    tol = 2e-5 if dtype == torch.float32 else 4e-2
    qw = torch.zeros(T, H, D).double()
    qw[..., :d] = turn(proj[:, :H * d].reshape(T, H, d))
    assert (q.double().cpu().view(T, H, D) - qw).abs().max().item() < tol
    kw = torch.zeros(T, Hkv, D).double()
    kw[..., :d] = turn(proj[:, H * d:(H + Hkv) * d].reshape(T, Hkv, d))
    v0 = (H + Hkv) * d
    for t in range(T):
        p = 11 + t
        pg = int(table[0, p // page])
        assert (kc[pg, :, p % page].double().cpu() - kw[t]).abs().max().item() < tol
        assert torch.equal(vc[pg, :, p % page, :e], proj[t, v0:v0 + Hkv * e].view(Hkv, e)) and (vc[pg, :, p % page, e:] == 0).all()


# ---- gated linear attention ------------------------------------------------------------------------------------------
def _gla_want(proj, low, w2t, bias, lens, H, d, e, tau, q_scale, states):
    """Per request, float64: outputs, and the states afterwards (lists of [H, d, e])."""
    out, t = [], 0
    states = [s.clone() for s in states]
    la = torch.nn.functional.logsigmoid(low.double() @ w2t.double() + bias.double()) / tau
    for s, n in enumerate(lens):
        for _ in range(n):
            q = proj[t, :H * d].double().view(H, d) * q_scale
            k = proj[t, H * d:2 * H * d].double().view(H, d)
            v = proj[t, 2 * H * d:2 * H * d + H * e].double().view(H, e)
            S = states[s] * torch.exp(la[t]).view(H, d, 1) + k[:, :, None] * v[:, None, :]
            states[s] = S
            out.append(torch.einsum("hde,hd->he", S, q).reshape(-1))
            t += 1
    return torch.stack(out), states


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,e,rank,tau,fade", [(2, 16, 24, 4, 16.0, 1.0), (3, 10, 7, 1, 1.0, 1.0), (1, 64, 64, 16, 16.0, 0.0), (2, 48, 33, 8, 2.0, -3.0),
                                                 (1, 96, 16, 20, 1.0, -12.0), (2, 130, 20, 5, 8.0, 2.0), (1, 256, 40, 3, 4.0, 0.0)])
def test_recurrence_token_by_token_and_in_chunks(dtype, H, d, e, rank, tau, fade):
    """Two steps of several requests in slots of their own, portions of 1 to 150 tokens (parts of a chunk, whole chunks,
    one token more), starting from states that are not zero; `fade` moves the decays from almost none to almost everything
    a token (a running sum of logarithms down to -400 inside a chunk).  Both forms, and both in one step."""
    from sandyrt_b200.csrc import ops

    g = torch.Generator().manual_seed(d + e)
    slots = torch.tensor([3, 0, 4, 1, 5], dtype=torch.int32, device=DEV)
    n_state = H * d * e
    for chunked_from in (0, 1, 8):
        state = torch.full((6, n_state + 9), 5.0, device=DEV)
        start = [torch.randn(H, d, e, generator=g).double() for _ in range(5)]
        for s in range(5):
            state[int(slots[s]), :n_state] = start[s].transpose(1, 2).reshape(-1).float().to(DEV)
        untouched = state[2].clone()
        want_states = start
        for lens in ([32, 1, 150, 7, 33], [1, 9, 8, 64, 31]):
            T = sum(lens)
            proj = torch.randn(T, 2 * H * d + 2 * H * e, generator=g).to(dtype)
            low = torch.randn(T, rank, generator=g)
            w2t = (torch.randn(rank, H * d, generator=g) / math.sqrt(rank)).contiguous()
            bias = torch.randn(H * d, generator=g) + fade
            q_start = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)
            out = torch.full((T, H * e), float("nan"), device=DEV)
            ops.gla_scan(proj.to(DEV), low.to(DEV), w2t.to(DEV), bias.to(DEV), state, q_start, slots, out, n_heads=H, qk_dim=d, v_dim=e,
                         tau=tau, q_scale=d ** -0.5, chunked_from=chunked_from, max_q_len=max(lens))
            want, want_states = _gla_want(proj, low, w2t, bias, lens, H, d, e, tau, d ** -0.5, want_states)
            size = want.abs().max().item()
            assert (out.double().cpu() - want).abs().max().item() < 3e-6 * max(size, 1.0), (chunked_from, lens)
            for s in range(5):
                got = state[int(slots[s]), :n_state].double().cpu().view(H, e, d).transpose(1, 2)
                assert (got - want_states[s]).abs().max().item() < 3e-6 * max(want_states[s].abs().max().item(), 1.0)
        assert torch.equal(state[2], untouched) and (state[:, n_state:] == 5.0).all()
