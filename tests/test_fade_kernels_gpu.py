"""Kernels of the recurrences with a decay per key channel, of the attention whose values are its keys, of several mixes of one
token shift and of several products in one launch, each alone against a plain float64 formula."""
import math

import pytest
import torch

from test_kernels_gpu import ATT_TOL, DEV, _paged_case

pytestmark = pytest.mark.gpu


# ---- the recurrences -------------------------------------------------------------------------------------------------
def _want(kind, q, k, v, la, beta, bonus, lens, states):
    """q, k, la [T, H, d], v [T, H, e] (float64, q scaled, heads already repeated); -> outputs and the states afterwards."""
    out, t = [], 0
    states = [s.clone() for s in states]
    for s, n in enumerate(lens):
        for _ in range(n):
            S = states[s]
            if kind == "bonus":
                kv = k[t][:, :, None] * v[t][:, None, :]
                o = torch.einsum("hde,hd->he", S + bonus[:, :, None] * kv, q[t])
                S = S * torch.exp(la[t])[:, :, None] + kv
            else:
                S = S * torch.exp(la[t])[:, :, None]
                u = v[t] if kind == "add" else beta[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
                S = S + k[t][:, :, None] * u[:, None, :]
                o = torch.einsum("hde,hd->he", S, q[t])
            states[s] = S
            out.append(o.reshape(-1))
            t += 1
    return torch.stack(out), states


SIZES = [(2, 2, 16, 24, 4, 0.0), (3, 1, 10, 7, 1, -2.0), (4, 2, 64, 64, 16, 0.0), (2, 1, 48, 33, 8, 3.0), (1, 1, 96, 16, 20, -5.0), (2, 2, 130, 20, 5, 1.0),
         (1, 1, 256, 40, 3, 0.0), (2, 1, 128, 128, 24, -1.0), (2, 2, 1, 1, 1, 0.0)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,decay", [("bonus", "exp"), ("delta", "softplus"), ("add", "logsigmoid"), ("delta", "logsigmoid"), ("bonus", "softplus")])
@pytest.mark.parametrize("H,Hq,d,e,rank,fade", SIZES)
def test_recurrence_token_by_token_and_in_chunks(dtype, kind, decay, H, Hq, d, e, rank, fade):
    """Two steps of several requests in slots of their own, portions of 1 to 150 tokens (parts of a chunk, whole chunks, one
    token more), starting from states that are not zero; `fade` moves the decays from almost none to almost everything a
    token.  Both forms, and both in one step."""
    from sandyrt_b200.csrc import ops

    g = torch.Generator().manual_seed(d + e + H)
    slots = torch.tensor([3, 0, 4, 1, 5], dtype=torch.int32, device=DEV)
    n_state = H * d * e
    up = lambda x: x.double().repeat_interleave(H // Hq, dim=1)
    for chunked_from in (0, 1, 8):
        state = torch.full((6, n_state + 9), 5.0, device=DEV)
        want_states = [torch.randn(H, d, e, generator=g).double() for _ in range(5)]
        for s in range(5):
            state[int(slots[s]), :n_state] = want_states[s].transpose(1, 2).reshape(-1).float().to(DEV)
        untouched = state[2].clone()
        for lens in ([32, 1, 150, 7, 33], [1, 9, 8, 64, 31]):
            T = sum(lens)
            q, k = torch.randn(T, Hq, d, generator=g), torch.randn(T, Hq, d, generator=g)
            if kind == "delta":                                    # the rule is stable for keys of at most unit length
                q, k = q / q.norm(dim=-1, keepdim=True), k / k.norm(dim=-1, keepdim=True) * 0.99
            q, k, v = q.to(dtype), k.to(dtype), torch.randn(T, H, e, generator=g).to(dtype)
            proj = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), torch.zeros(T, 5, dtype=dtype)], 1).to(DEV)
            low = torch.randn(T, rank + 3, generator=g)
            w2t = (torch.randn(rank, H * d, generator=g) / math.sqrt(rank)).contiguous()
            bias, a_log = torch.randn(H * d, generator=g) + fade, torch.randn(H, generator=g)
            bonus, beta = torch.randn(H * d, generator=g), torch.randn(T, H + 2, generator=g)
            tanh = kind == "bonus"
            lo = low[:, :rank].double()
            z = ((torch.tanh(lo) if tanh else lo) @ w2t.double() + bias.double()).view(T, H, d)
            la = {"exp": lambda: -torch.exp(z), "softplus": lambda: -torch.exp(a_log.double())[None, :, None] * torch.nn.functional.softplus(z),
                  "logsigmoid": lambda: torch.nn.functional.logsigmoid(z) / 4.0}[decay]()
            q_start = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32, device=DEV)
            out = torch.full((T, H * e), float("nan"), device=DEV)
            dev = lambda t: t.to(DEV)
            ops.fade_scan(proj, dev(low)[:, :rank], dev(w2t), dev(bias), state, q_start, slots, out, n_heads=H, n_qk_heads=Hq, qk_dim=d, v_dim=e,
                          q_scale=0.5, kind=kind, decay=decay, tau=4.0, tanh_low=tanh, a_log=dev(a_log), bonus=dev(bonus),
                          beta=dev(beta)[:, :H], chunked_from=chunked_from, max_q_len=max(lens))
            want, want_states = _want(kind, up(q) * 0.5, up(k), v.double(), la, torch.sigmoid(beta[:, :H].double()), bonus.double().view(H, d), lens,
                                      want_states)
            size = max(want.abs().max().item(), 1.0)
            assert (out.double().cpu() - want).abs().max().item() < 6e-6 * size, (chunked_from, lens)
            for s in range(5):
                got = state[int(slots[s]), :n_state].double().cpu().view(H, e, d).transpose(1, 2)
                assert (got - want_states[s]).abs().max().item() < 6e-6 * max(want_states[s].abs().max().item(), 1.0)
        assert torch.equal(state[2], untouched) and (state[:, n_state:] == 5.0).all()


def test_decays_beyond_what_a_float_holds():
    """Channels that fade to nothing in a token (exponents of minus thousands) beside channels that do not fade, in chunks: no
    overflow, no NaN, and the slow channels keep their exact sums."""
    from sandyrt_b200.csrc import ops

    H, d, e, T = 1, 32, 16, 70
    g = torch.Generator().manual_seed(2)
    proj = torch.randn(T, 3 * 32, generator=g)[:, :2 * d + e].contiguous()
    low, w2t = torch.zeros(T, 1), torch.zeros(1, d)
    bias = torch.tensor([-30.0, 9.0, 100.0, -2.0] * 8)
    la = -torch.exp(bias.double()).expand(T, d)[:, None]
    for chunked_from in (0, 1):
        state, out = torch.zeros(1, d * e, device=DEV), torch.empty(T, e, device=DEV)
        ops.fade_scan(proj.to(DEV), low.to(DEV), w2t.to(DEV), bias.to(DEV), state, torch.tensor([0, T], dtype=torch.int32, device=DEV),
                      torch.zeros(1, dtype=torch.int32, device=DEV), out, n_heads=1, qk_dim=d, v_dim=e, q_scale=1.0, kind="bonus", decay="exp",
                      bonus=torch.ones(d, device=DEV), chunked_from=chunked_from, max_q_len=T)
        want, _ = _want("bonus", proj[:, None, :d].double(), proj[:, None, d:2 * d].double(), proj[:, None, 2 * d:].double(), la, None,
                        torch.ones(1, d).double(), [T], [torch.zeros(1, d, e).double()])
        assert (out.double().cpu() - want).abs().max().item() < 6e-6 * want.abs().max().item()


# ---- attention ---------------------------------------------------------------------------------------------------------
def _att_want(case, H, Hkv, scale, window, cap, sink, gate, out_gate):
    outs, t = [], 0
    for s, (before, n) in enumerate(case["seqs"]):
        k, v, q = case["dense_k"][s].double(), case["dense_v"][s].double(), case["qs"][s].double()
        for i in range(n):
            pos = before + i
            lo = max(0, pos - window + 1) if window else 0
            row = []
            for h in range(H):
                kh = h // (H // Hkv)
                sc = (k[lo:pos + 1, kh] @ q[i, h]) * scale
                p = torch.exp(cap * torch.tanh(sc / cap) if cap else sc)
                o = (p @ v[lo:pos + 1, kh]) / (p.sum() + (math.exp(float(sink[h])) if sink is not None else 0.0))
                if gate is not None:
                    D = o.numel()
                    o = o * torch.sigmoid(gate[t, h * D:(h + 1) * D])
                row.append(o * (float(out_gate[t, h]) if out_gate is not None else 1.0))
            outs.append(torch.cat(row))
            t += 1
    return torch.stack(outs)


# (H, Hkv, D, page, window, capped and gated | sinks and a factor)
ATT = [(4, 2, 64, 16, 40, True), (12, 4, 64, 16, 0, True), (6, 2, 48, 8, 17, True), (8, 2, 128, 16, 33, True), (10, 2, 128, 16, 45, False), (16, 2, 128, 16, 0, False),
       (4, 4, 64, 16, 70, False), (6, 3, 32, 8, 1, False), (4, 1, 128, 32, 129, False)]


@pytest.mark.parametrize("H,Hkv,D,page,window,capped", ATT)
@pytest.mark.parametrize("how", ["prompt", "prompt tcgen05", "decode, rows", "general", "general float32"])
def test_caps_sinks_gates_and_windows_together(how, H, Hkv, D, page, window, capped):
    """What the two attentions of this design ask of a kernel at once: a cap, a window and a gate by element; or sinks of
    their own per head, a window and a factor."""
    from sandyrt_b200.csrc import ops

    if how == "prompt tcgen05" and D != 64:
        pytest.skip("heads of 64")
    dtype = torch.float32 if how == "general float32" else torch.bfloat16
    seqs = [(699, 1), (0, 1), (63, 1), (300, 1), (max(0, window - 1), 1), (window, 1), (window + 1, 1)]
    if how.startswith("prompt"):
        seqs = [(0, 150), (520, 70), (17, 70), (0, 1), (640, 3), (window, 2)]
    case = _paged_case(dtype, H, Hkv, D, page, seqs, seed=D + H)
    T = case["q"].shape[0]
    g = torch.Generator().manual_seed(H)
    gate = torch.randn(T, H * D + 16, generator=g).to(dtype).to(DEV)[:, 8:8 + H * D] if capped else None
    sink = None if capped else torch.randn(H, generator=g).mul(2).to(DEV)
    factor = None if capped else (torch.rand(T, H, generator=g) + 0.5).to(DEV)
    cap, scale = (1.5, 2.0 / math.sqrt(D)) if capped else (0.0, 1.0 / math.sqrt(D))
    out = torch.full_like(case["q"], float("nan"))
    kw = dict(n_heads=H, scale=scale, window=window)
    if capped:
        kw.update(softcap=cap, elem_gate=gate)
    else:
        kw.update(sink=sink, out_gate=factor)
    if how.startswith("prompt"):
        q_start = torch.tensor([0] + list(torch.tensor([n for _, n in seqs]).cumsum(0)), dtype=torch.int32, device=DEV)
        kv_before = torch.tensor([b for b, _ in seqs], dtype=torch.int32, device=DEV)
        ops.prefill_attention(case["q"], case["kc"], case["vc"], case["table"], q_start, kv_before, out, max_q_len=150, tc=how.endswith("tcgen05"), **kw)
    else:
        args = (case["q"], case["kc"], case["vc"], case["table"], case["tok_seq"], case["tok_pos"], out)
        if how == "decode, rows":
            ops.decode_attention_shared(*args, splits=2, **kw)
        else:
            ops.paged_attention(*args, **kw)
    ops.check_kernel_status(DEV)
    cpu = lambda t: None if t is None else t.double().cpu()
    want = _att_want(case, H, Hkv, scale, window, cap, cpu(sink), cpu(gate), cpu(factor))
    assert (out.double().cpu() - want).abs().max().item() < ATT_TOL[dtype] * 1.5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,Hkv,d,rot", [(4, 2, 16, 8), (3, 1, 20, 20), (2, 2, 64, 32)])
def test_values_are_the_keys_before_they_turn(dtype, H, Hkv, d, rot):
    """One projection feeds both planes of the cache: the key plane turned, cosine and sine times a factor that the rest of the
    head does not get, the value plane as projected; and a factor per head and token of its own."""
    from sandyrt_b200.csrc import ops

    T, page, D, m = 23, 8, -(-d // 16) * 16, 1.3
    g = torch.Generator().manual_seed(d)
    proj = torch.randn(T, (H + Hkv) * d + 5, generator=g).to(dtype).to(DEV)
    pos = torch.arange(11, 11 + T, dtype=torch.int32, device=DEV)
    arena = torch.full((8, 2, Hkv, page, D), 7.0, dtype=dtype, device=DEV)
    kc, vc = arena[:, 0], arena[:, 1]
    table = torch.tensor([[5, 3, 1, 0, 2, 4]], dtype=torch.int32, device=DEV)
    seq = torch.zeros(T, dtype=torch.int32, device=DEV)
    freq = torch.tensor([30.0 ** (-2 * i / rot) for i in range(rot // 2)], device=DEV)
    q, factor = torch.full((T, H * D), float("nan"), dtype=dtype, device=DEV), torch.zeros(T, H, device=DEV)
    ops.attention_prepare(proj, kc, vc, table, seq, pos, q, n_heads=H, qk_dim=d, v_dim=d, freq=freq, interleaved=True, rot_scale=m,
                          values_are_keys=True, head_scale=(factor, 0.7))
    ops.check_kernel_status(DEV)
    assert (factor == 0.7).all()

    def turn(x):
        x = x.double().cpu().clone()
        y = x.clone()
        for i in range(rot // 2):
            a = torch.arange(11, 11 + T).double() * float(freq[i])
            c, s = m * torch.cos(a)[:, None], m * torch.sin(a)[:, None]
            y[:, :, 2 * i] = x[:, :, 2 * i] * c - x[:, :, 2 * i + 1] * s
            y[:, :, 2 * i + 1] = x[:, :, 2 * i + 1] * c + x[:, :, 2 * i] * s
        return y

    tol = 2e-5 if dtype == torch.float32 else 5e-2
    assert (q.double().cpu().view(T, H, D)[..., :d] - turn(proj[:, :H * d].reshape(T, H, d))).abs().max().item() < tol
    k = proj[:, H * d:(H + Hkv) * d].reshape(T, Hkv, d)
    turned = turn(k)
    for t in range(T):
        pg, at = int(table[0, (11 + t) // page]), (11 + t) % page
        assert (kc[pg, :, at, :d].double().cpu() - turned[t]).abs().max().item() < tol
        assert torch.equal(vc[pg, :, at, :d], k[t]) and (vc[pg, :, at, d:] == 0).all() and (kc[pg, :, at, d:] == 0).all()


# ---- token shift and products ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,n_mix", [(48, 5), (100, 3), (768, 5), (1536, 2), (5000, 5)])
def test_several_mixes_of_one_token_shift(dtype, width, n_mix):
    from sandyrt_b200.csrc import ops

    g = torch.Generator().manual_seed(width)
    lens, slots = [5, 1, 9, 1], [2, 0, 3, 1]
    T = sum(lens)
    x, gain, mix = torch.randn(T, width, generator=g), torch.randn(width, generator=g) + 1, torch.rand(n_mix, width, generator=g)
    state = torch.randn(4, width + 3, generator=g)
    starts = [0, 5, 6, 15, 16]
    h = x.double() / torch.sqrt((x.double() ** 2).mean(-1, keepdim=True) + 1e-5) * gain.double()
    want = torch.empty(T, n_mix * width).double()
    for s, n in enumerate(lens):
        for i in range(n):
            t = starts[s] + i
            before = h[t - 1] if i else state[slots[s], :width].double()
            want[t] = torch.cat([h[t] + (before - h[t]) * mix[j].double() for j in range(n_mix)])
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    out, st = torch.full((T, n_mix * width), float("nan"), dtype=dtype, device=DEV), state.to(DEV)
    ops.rmsnorm_shift(x.to(DEV), gain.to(DEV), mix.to(DEV), st, i32([s for s, n in enumerate(lens) for _ in range(n)]), i32(starts), i32(slots),
                      out, eps=1e-5)
    assert (out.double().cpu() - want).abs().max().item() < (2e-5 if dtype == torch.float32 else 4e-2)
    for s, n in enumerate(lens):
        assert (st[slots[s], :width].double().cpu() - h[starts[s] + n - 1]).abs().max().item() < 2e-5
    assert torch.equal(st[:, width:].cpu(), state[:, width:])


@pytest.mark.parametrize("M", [1, 8, 16, 17, 33, 64])
@pytest.mark.parametrize("groups,N,K", [(4, 48, 96), (4, 768, 768), (3, 16, 8), (2, 1040, 200)])
def test_products_of_one_shape_in_one_launch(M, groups, N, K):
    """Every group reads its own columns of the input; the same bits as one product at a time where both take the same form."""
    from sandyrt_b200.csrc import ops

    g = torch.Generator().manual_seed(N + M)
    a = torch.randn(M, groups * K, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(groups * N, K, generator=g) / math.sqrt(K)).to(torch.bfloat16).to(DEV)
    for dt in (torch.float32, torch.bfloat16):
        out = torch.full((M, groups * N), float("nan"), dtype=dt, device=DEV)
        ops.gemm_skinny_groups(a, w, out, n_groups=groups)
        want = torch.cat([a[:, i * K:(i + 1) * K].double() @ w[i * N:(i + 1) * N].double().t() for i in range(groups)], 1)
        assert (out.double() - want).abs().max().item() < (2e-5 * math.sqrt(K) if dt == torch.float32 else 4e-2)
