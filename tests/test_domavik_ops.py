"""Mechanisms of the Domavik decoder one by one against the plain statements of ``domavik_oracle``: window attention with
kept tokens and a distance bias, the two gated recurrences, and the row operations around them.  The same cases run on the
framework's CPU path, its 32-bit CUDA kernels and its bf16 CUDA kernels."""
import math

import domavik_oracle as O
import pytest
import torch

from siirl_b200.ops import rows as R
from siirl_b200.ops.recurrence import PortionPlan, RecurrenceSpec, empty_state, recurrence_decode, recurrence_prefill
from siirl_b200.ops.window_attention import QueryTiles, WindowSpec, window_attention

GPU = pytest.mark.gpu
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    """Thousands of tiny CPU operations: thread pools only slow them down."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def close(got, want, dtype, what="", rel=None):
    got, want = got.detach().double().cpu(), want.double()
    tol = rel if rel is not None else (2e-5 if dtype == torch.float32 else 1.5e-2)
    err = (got - want).abs().max().item()
    lim = tol * max(want.abs().max().item(), 1e-6)
    assert err <= lim, f"{what}: {err:.3e} > {lim:.3e}"


def finish(device):
    if device == "cuda":
        from siirl_b200.ops import lib
        torch.cuda.synchronize()
        lib.check_status()


# ---- window attention ------------------------------------------------------------------------------------------------------
ATT = {  # heads, kv_heads, dk, dv, window, keep_first
    "group3": (6, 2, 32, 24, 70, 5), "one_head": (1, 1, 16, 40, 9, 3), "page_window": (4, 2, 64, 64, 64, 64),
    "wide": (4, 4, 128, 96, 130, 65), "no_sink": (2, 1, 48, 48, 33, 0), "very_wide": (2, 1, 192, 256, 100, 20),
    "odd": (3, 3, 20, 13, 50, 7), "window1": (2, 2, 32, 32, 1, 2), "whole_group": (8, 1, 72, 120, 77, 66),
    "many_heads": (20, 2, 64, 32, 90, 1), "sink_over_window": (2, 2, 32, 32, 20, 130),
}


def att_case(name, T, seed=0):
    """Random rows with queries that single out keys at the edges of what they see, and just beyond."""
    H, G, dk, dv, w, kf = ATT[name]
    g = torch.Generator().manual_seed(seed)
    q = torch.randn(T, H, dk, generator=g)
    k = torch.randn(T, G, dk, generator=g)
    v = torch.randn(T, G, dv, generator=g)
    scale = 1.3 * dk ** -0.5
    for i in range(T):
        spots = [i - w + 1, i - w, kf - 1, kf, i, i - 64, i // 64 * 64]
        j = spots[i % len(spots)]
        if 0 <= j <= i:
            for h in range(H):
                kk = k[j, h // (H // G)]
                # score well above the others and above the bias of the distance
                q[i, h] = kk * ((12.0 + 2.0 ** (-8.0 * (h + 1) / H) * (i - j)) / (scale * (kk * kk).sum()))
    r = lambda t: t.bfloat16().double()  # noqa: E731
    return r(q), r(k), r(v), scale


class Pages:
    """A cache with scattered blocks, one table row per slot."""

    def __init__(self, spec, slots, max_len, dtype, device, seed=3):
        g = torch.Generator().manual_seed(seed)
        nb = (max_len + 63) // 64
        order = torch.randperm(slots * nb + 3, generator=g)[: slots * nb].to(torch.int32)
        self.table = order.view(slots, nb).to(device)
        # blocks hold what earlier sequences left: finite values that must not matter
        self.cache = (torch.randn(slots * nb + 3, spec.block_elems, generator=g) * 30).to(dtype).to(device)


def att_spec(name, scale, pad=8, out_scale=1.0):
    H, G, dk, dv, w, kf = ATT[name]
    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    qo = pad
    ko = qo + up(H * dk)
    vo = ko + up(G * dk)
    spec = WindowSpec(H, G, dk, dv, qo, ko, vo, scale, w, kf, 8.0, out_scale)
    return spec, vo + up(G * dv) + 8


def pack(spec, width, q, k, v, dtype, device):
    T = q.shape[0]
    x = torch.full((T, width), 7.0, dtype=torch.float64)
    for off, t in ((spec.q_off, q), (spec.k_off, k), (spec.v_off, v)):
        x[:, off:off + t[0].numel()] = t.reshape(T, -1)
    return x.to(dtype).to(device)


def run_portions(spec, x, pages, slot, cuts, out, simt=False):
    at = 0
    for n in cuts:
        dev = x.device
        pos = torch.arange(at, at + n, dtype=torch.int32, device=dev)
        ids = torch.full((n,), slot, dtype=torch.int32, device=dev)
        window_attention(spec, x[at:at + n], ids, pos, pages.table, pages.cache, out[at:at + n], 16,
                         tiles=QueryTiles([n], [at], [slot], dev), simt=simt)
        at += n


def run_single(spec, x, pages, slot, at, out):
    """One decode row in a batch with idle slots."""
    S, dev = pages.table.shape[0], x.device
    rows = torch.zeros(S, x.shape[1], dtype=x.dtype, device=dev)
    rows[slot] = x[at]
    ids = torch.full((S,), -1, dtype=torch.int32, device=dev)
    ids[slot] = slot
    pos = torch.zeros(S, dtype=torch.int32, device=dev)
    pos[slot] = at
    lens = torch.zeros(S, dtype=torch.int32, device=dev)
    lens[slot] = at + 1
    o = torch.full((S, out.shape[1]), 5.0, dtype=x.dtype, device=dev)
    window_attention(spec, rows, ids, pos, pages.table, pages.cache, o, 16, seq_lens=lens)
    out[at] = o[slot]
    idle = [s for s in range(S) if s != slot]
    assert o[idle, 16:16 + spec.heads * spec.vdim].abs().max().item() == 0


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(ATT))
def test_window_attention_prompts_portions_and_single_tokens(name, device, dtype):
    T = 203
    q, k, v, scale = att_case(name, T)
    H, _, _, dv, w, kf = ATT[name]
    want = O.window_attention_fast(q, k, v, scale, w, kf).reshape(T, -1) * 0.75
    spec, width = att_spec(name, scale, out_scale=0.75)
    x = pack(spec, width, q, k, v, dtype, device)
    for cuts in ([T], [2, 62, 64, 1, 66, 8], [128, 75]):
        pages = Pages(spec, 3, 256, dtype, device)
        out = torch.full((T, 16 + (H * dv + 7) // 8 * 8), 9.0, dtype=dtype, device=device)
        run_portions(spec, x, pages, 1, cuts, out)
        finish(device)
        close(out[:, 16:16 + H * dv], want, dtype, f"portions {cuts}")
        assert (out[:, :16] == 9).all()
    pages = Pages(spec, 3, 256, dtype, device)
    out = torch.zeros(T, 16 + (H * dv + 7) // 8 * 8, dtype=dtype, device=device)
    run_portions(spec, x, pages, 2, [97], out)
    for at in range(97, T):
        run_single(spec, x, pages, 2, at, out)
    finish(device)
    close(out[:, 16:16 + H * dv], want, dtype, "single tokens")


@pytest.mark.parametrize("device,dtype", WHERE)
def test_window_attention_of_a_long_context_in_chunks(device, dtype):
    """A window of more than 1024 tokens: decoding splits the visible blocks over several work items."""
    ATT["long"] = (4, 2, 64, 64, 1500, 70)
    T = 2300 if device == "cuda" else 300
    q, k, v, scale = att_case("long", T)
    spec, width = att_spec("long", scale)
    x = pack(spec, width, q, k, v, dtype, device)
    pages = Pages(spec, 2, T + 64, dtype, device)
    out = torch.zeros(T, 16 + 256, dtype=dtype, device=device)
    run_portions(spec, x, pages, 0, [T - 9], out)
    for at in range(T - 9, T):
        run_single(spec, x, pages, 0, at, out)
    finish(device)
    want = O.window_attention_fast(q, k, v, scale, 1500, 70).reshape(T, -1)
    close(out[:, 16:], want, dtype)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_window_attention_of_unequal_sequences_in_one_batch(device, dtype):
    name, lens, starts = "group3", [1, 130, 64, 7], [0, 65, 2, 70]
    spec = None
    xs, wants, pages = [], [], None
    for i, (n, st) in enumerate(zip(lens, starts)):
        q, k, v, scale = att_case(name, st + n, seed=i)
        if spec is None:
            spec, width = att_spec(name, scale)
            pages = Pages(spec, 4, 256, dtype, device)
        H, _, _, dv, w, kf = ATT[name]
        wants.append(O.window_attention_fast(q, k, v, scale, w, kf).reshape(st + n, -1)[st:])
        x = pack(spec, width, q, k, v, dtype, device)
        if st:
            scratch = torch.zeros(st, 16 + H * dv, dtype=dtype, device=device)
            run_portions(spec, x[:st], pages, 3 - i, [st], scratch)
        xs.append(x[st:])
    slots = [3, 2, 1, 0]
    ids = torch.cat([torch.full((n,), s, dtype=torch.int32) for n, s in zip(lens, slots)]).to(device)
    pos = torch.cat([torch.arange(st, st + n, dtype=torch.int32) for n, st in zip(lens, starts)]).to(device)
    x = torch.cat(xs)
    out = torch.zeros(x.shape[0], 16 + H * dv, dtype=dtype, device=device)
    window_attention(spec, x, ids, pos, pages.table, pages.cache, out, 16,
                     tiles=QueryTiles(lens, starts, slots, torch.device(device)))
    finish(device)
    close(out[:, 16:], torch.cat(wants), dtype)


def test_the_attention_cases_show_every_edge():
    """The inputs above tell a window, a kept range or a bias that is slightly off from the right one."""
    for name in ("group3", "one_head", "page_window", "no_sink"):
        q, k, v, scale = att_case(name, 203)
        w, kf = ATT[name][4:]
        right = O.window_attention_fast(q, k, v, scale, w, kf)
        wrong = [O.window_attention_fast(q, k, v, scale, w + 1, kf), O.window_attention_fast(q, k, v, scale, w - 1, kf),
                 O.window_attention_fast(q, k, v, scale, w, kf + 1)]
        if kf:
            wrong.append(O.window_attention_fast(q, k, v, scale, w, kf - 1))
        for other in wrong:
            assert (right - other).abs().max() > 0.15 * right.abs().max()
        assert torch.allclose(right, O.window_attention(q, k, v, scale, w, kf), atol=1e-12)


# ---- recurrences -----------------------------------------------------------------------------------------------------------
REC = {  # gate, heads, dk, dv
    "channel": ("channel", 3, 32, 48), "channel_small": ("channel", 1, 8, 16), "channel_wide": ("channel", 2, 128, 128),
    "channel_48": ("channel", 4, 48, 32), "channel_ragged": ("channel", 2, 40, 24), "channel_odd": ("channel", 2, 21, 19),
    "channel_256": ("channel", 1, 256, 200), "head": ("head", 3, 32, 48), "head_one": ("head", 1, 16, 8),
    "head_wide": ("head", 2, 128, 128), "head_ragged": ("head", 5, 24, 40), "head_odd": ("head", 2, 19, 21),
    "head_96": ("head", 2, 96, 176),
}


def rec_case(name, T, hard=False, seed=0):
    gate, H, dk, dv = REC[name]
    rank = 5 if name == "channel_odd" else 8
    up = lambda n: (n + 7) // 8 * 8  # noqa: E731
    g = torch.Generator().manual_seed(seed)
    n = lambda *s: torch.randn(*s, generator=g).bfloat16().double()  # noqa: E731
    off, at = {}, 8
    widths = dict(q=H * dk, k=H * dk, v=H * dv, g=H * dv)
    widths.update(dict(e=rank) if gate == "channel" else dict(e=H, f=H))
    cols = {}
    for key, wd in widths.items():
        off[key], at = at, at + up(wd)
        cols[key] = n(T, wd)
    wts = {"norm": (1 + 0.2 * n(H * dv if gate == "head" else dv)).bfloat16().double()}
    tau, cap, eps = (1.0 if hard else 6.0), 7.0, 1e-3
    if gate == "channel":
        wts["w2"], wts["b_e"] = n(H * dk, rank), (n(H * dk) * (6 if hard else 1)).bfloat16().double()
    else:
        spread = 12.0 if hard else 1.5
        cols["e"], cols["f"] = (cols["e"] * spread).bfloat16().double(), (cols["f"] * spread).bfloat16().double()
        wts["b_e"], wts["b_f"] = n(H), (n(H) + 2).bfloat16().double()
    x = torch.full((T, at + 8), 3.0, dtype=torch.float64)
    for key, t in cols.items():
        x[:, off[key]:off[key] + t.shape[1]] = t
    spec = RecurrenceSpec(gate, H, dk, dv, off["q"], off["k"], off["v"], off["g"], off["e"], off.get("f", 0),
                          rank if gate == "channel" else 0, tau, cap, eps, 0.6,
                          "silu" if gate == "channel" else "sigmoid", gate == "head")
    q = cols["q"].view(T, H, dk) * dk ** -0.5
    k, v, og = cols["k"].view(T, H, dk), cols["v"].view(T, H, dv), cols["g"]
    if gate == "channel":
        z = (cols["e"] @ wts["w2"].T + wts["b_e"]).view(T, H, dk)
        o, S = O.gated_linear(q, k, v, z, tau)
        y = (O.rms(o, eps) * wts["norm"]).reshape(T, -1) * og * torch.sigmoid(og) * 0.6
        state = {"S": S.transpose(1, 2)}
    else:
        o, (S, nn, m) = O.matrix_memory(q, k, v, cols["e"] + wts["b_e"], cols["f"] + wts["b_f"], cap)
        y = O.rms(o, eps).reshape(T, -1) * wts["norm"] * torch.sigmoid(og) * 0.6
        state = {"S": torch.cat([S.transpose(1, 2), nn[:, None]], 1), "m": m}
    return spec, x, wts, y, state


def dirty_state(spec, slots, device):
    """Slots as an earlier sequence left them."""
    st = empty_state(spec, slots, device)
    for t in st.values():
        t.fill_(11.0)
    return st


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("hard", [False, True], ids=["plain", "hard"])
@pytest.mark.parametrize("name", list(REC))
def test_recurrence_prompts_portions_and_single_tokens(name, hard, device, dtype):
    T = 51
    spec, x, wts, want, state = rec_case(name, T, hard)
    H, dv = spec.heads, spec.vdim
    xd = x.to(dtype).to(device)
    wd = {k: t.to(dtype).to(device).contiguous() for k, t in wts.items()}
    width = 8 + (H * dv + 7) // 8 * 8
    tol = 1e-4 if dtype == torch.float32 else 1e-2

    def check(out, st, what):
        finish(device)
        close(out[:, 8:8 + H * dv], want, dtype, what, tol)
        for key, t in state.items():
            # the state is 32-bit whatever the format of the rows
            close(st[key][2], t, torch.float32, f"{what}: state {key}", 5e-4)

    for cuts in ([T], [2, 16, 17, 16], [33, 18]):
        for stepwise in ((False, True) if device == "cuda" else (False,)):
            st = dirty_state(spec, 3, device)
            out = torch.zeros(T, width, dtype=dtype, device=device)
            at = 0
            for n in cuts:
                recurrence_prefill(spec, xd[at:at + n], wd, st, PortionPlan([n], [at], [2], torch.device(device)),
                                   out[at:at + n], 8, stepwise=stepwise)
                at += n
            check(out, st, f"portions {cuts} stepwise {stepwise}")
    st = dirty_state(spec, 3, device)
    out = torch.zeros(T, width, dtype=dtype, device=device)
    for t in range(T):      # token by token from the first, beside idle rows
        rows = xd[t:t + 1].expand(3, -1).contiguous()
        slots = torch.tensor([-1, 2, -1], dtype=torch.int32, device=device)
        pos = torch.tensor([0, t, 0], dtype=torch.int32, device=device)
        o = torch.full((3, width), 4.0, dtype=dtype, device=device)
        recurrence_decode(spec, rows, wd, st, slots, pos, o, 8)
        out[t] = o[1]
        assert o[[0, 2], 8:8 + H * dv].abs().max().item() == 0
    check(out, st, "single tokens")
    assert (st["S"][:2] == 11).all()


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("gate", ["channel", "head"])
def test_recurrence_of_unequal_sequences_in_one_batch(gate, device, dtype):
    lens = [1, 50, 16, 33, 3]
    cases = [rec_case(gate, n, seed=i) for i, n in enumerate(lens)]
    spec = cases[0][0]
    wts = cases[0][2]
    # one set of weights: recompute the expectation of every sequence alone
    wd = {k: t.to(dtype).to(device).contiguous() for k, t in wts.items()}
    HV = spec.heads * spec.vdim
    st = dirty_state(spec, 5, device)
    x = torch.cat([c[1] for c in cases]).to(dtype).to(device)
    out = torch.zeros(x.shape[0], HV, dtype=dtype, device=device)
    slots = [4, 0, 2, 1, 3]
    recurrence_prefill(spec, x, wd, st, PortionPlan(lens, [0] * 5, slots, torch.device(device)), out, 0)
    at = 0
    for n, s in zip(lens, slots):
        one = torch.zeros(n, HV, dtype=dtype, device=device)
        st1 = dirty_state(spec, 1, device)
        recurrence_prefill(spec, x[at:at + n], wd, st1, PortionPlan([n], [0], [0], torch.device(device)), one, 0)
        assert torch.equal(one, out[at:at + n])
        assert torch.equal(st1["S"][0], st["S"][s])
        at += n
    finish(device)


@pytest.mark.parametrize("device,dtype", [WHERE[1], WHERE[2]])
def test_long_matrix_memory_prompt_scans_its_gates_in_blocks(device, dtype):
    """Longer than one block of the gate scan (1024 tokens), in one portion and in two."""
    spec, x, wts, want, state = rec_case("head_one", 2100)
    xd, wd = x.to(dtype).to(device), {k: t.to(dtype).to(device).contiguous() for k, t in wts.items()}
    for cuts in ([2100], [1025, 1075]):
        st = dirty_state(spec, 1, device)
        out = torch.zeros(2100, 8, dtype=dtype, device=device)
        at = 0
        for n in cuts:
            recurrence_prefill(spec, xd[at:at + n], wd, st, PortionPlan([n], [at], [0], torch.device(device)),
                               out[at:at + n], 0)
            at += n
        finish(device)
        close(out, want, dtype, str(cuts), 1e-3 if dtype == torch.float32 else 1e-2)
        close(st["m"][0], state["m"], torch.float32, "m", 1e-4)


# ---- row operations ----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("W", [8, 50, 320, 1024, 1028, 4096, 5000])
def test_add_norm_and_scaled_embedding(W, device, dtype):
    g = torch.Generator().manual_seed(W)
    T = 9
    h = torch.randn(T, W, generator=g).double() * 2 + 0.7
    delta = torch.randn(T, W, generator=g).to(dtype)
    w = (1 + 0.1 * torch.randn(W, generator=g)).to(dtype)
    for kind in ("layer_norm", "rms_norm"):
        for d in (None, delta):
            hd = h.float().to(device)
            y = R.add_norm(hd, None if d is None else d.to(device), w.to(device), 1e-3, kind)
            s = h.float().double() if d is None else h.float().double() + d.double()
            close(hd, s, torch.float32, "stream", 1e-6)
            want = O.layer_norm(s, w.double(), 1e-3) if kind == "layer_norm" else O.rms(s, 1e-3) * w.double()
            close(y, want, dtype, kind, 2e-6 * 10 if dtype == torch.float32 else 5e-3)
    table = torch.randn(37, W, generator=g).to(dtype)
    ids = torch.randint(0, 37, (T,), generator=g)
    e = R.embed_scaled(ids.to(device), table.to(device), 2.5)
    assert e.dtype == torch.float32
    close(e, table.double()[ids] * 2.5, torch.float32, "embedding", 1e-6)
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
def test_gated_activation_and_soft_cap(device, dtype):
    g = torch.Generator().manual_seed(1)
    for inner in (8, 12, 200, 33):
        gu = (torch.randn(7, 2 * inner, generator=g) * 3).to(dtype)
        a, b = gu.double().chunk(2, -1)
        close(R.gated_act(gu.to(device), "gelu_tanh"), O.gelu_tanh(a) * b, dtype, "gelu")
        close(R.gated_act(gu.to(device), "silu"), a * torch.sigmoid(a) * b, dtype, "silu")
    z = torch.randn(5, 77, generator=g) * 40
    close(R.softcap_(z.clone().to(device), 11.0), 11 * torch.tanh(z.double() / 11), torch.float32, "cap")
    finish(device)


@GPU
@pytest.mark.parametrize("shape", [(1, 5, 7), (70, 130, 33), (64, 64, 16), (129, 8, 500)])
def test_simt_matrix_product(shape):
    M, N, K = shape
    g = torch.Generator().manual_seed(2)
    a, b = torch.randn(M, K, generator=g), torch.randn(N, K, generator=g)
    close(R.gemm_simt(a.cuda(), b.cuda(), torch.float32), a.double() @ b.double().T, torch.float32, rel=1e-6 * math.sqrt(K) * 3)
    ab, bb = a.bfloat16(), b.bfloat16()
    for out in (torch.float32, torch.bfloat16):
        close(R.gemm_simt(ab.cuda(), bb.cuda(), out), ab.double() @ bb.double().T, out)
