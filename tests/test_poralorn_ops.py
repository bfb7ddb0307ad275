"""Mechanisms of the Poralorn decoder one by one against the plain statements of ``poralorn_oracle``: latent attention
(expanded and absorbed forms, paged latents), per-head products, the gated residual update, the entry of a loop's pass and
the activations.  The same cases run on the framework's CPU path, its 32-bit CUDA kernels and its bf16 CUDA kernels."""
import math

import poralorn_oracle as O
import pytest
import torch

from siirl_b200.ops import rows as R
from siirl_b200.ops.dense import linear_partial
from siirl_b200.ops.latent_attention import LatentPlan, LatentSpec, head_product, latent_attention

GPU = pytest.mark.gpu
CUDA = [pytest.param(torch.float32, id="cuda-f32", marks=GPU), pytest.param(torch.bfloat16, id="cuda-bf16", marks=GPU)]
WHERE = [pytest.param("cpu", torch.float32, id="cpu"), pytest.param("cuda", torch.float32, id="cuda-f32", marks=GPU),
         pytest.param("cuda", torch.bfloat16, id="cuda-bf16", marks=GPU)]


@pytest.fixture(autouse=True, scope="module")
def _one_thread():
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def close(got, want, dtype, what="", rel=None):
    got, want = got.detach().double().cpu(), want.double()
    tol = rel if rel is not None else (3e-5 if dtype == torch.float32 else 2e-2)
    err = (got - want).abs().max().item()
    lim = tol * max(want.abs().max().item(), 1e-6)
    assert err <= lim, f"{what}: {err:.3e} > {lim:.3e}"


def finish(device):
    if device == "cuda":
        from siirl_b200.ops import lib
        torch.cuda.synchronize()
        lib.check_status()


# ---- latent attention ------------------------------------------------------------------------------------------------------
LAT = {  # heads, dim, vdim, rank, output gate
    "mixed": (3, 24, 40, 48, True), "one": (1, 16, 8, 16, True), "equal": (2, 64, 64, 64, False),
    "wide": (16, 128, 128, 512, True), "three_chunks": (6, 48, 32, 192, True), "two_warps": (40, 32, 24, 136, True),
    "two_groups": (72, 16, 16, 64, False), "three_groups": (130, 8, 8, 24, True), "tall": (4, 192, 256, 320, True),
    "odd": (3, 13, 11, 21, True), "long_rank": (2, 32, 32, 640, True), "tight": (33, 16, 16, 512, True),
}
GAIN, EPS = 0.75, 1e-3
r16 = lambda t: t.bfloat16().double()  # noqa: E731


class Case:
    """Projected rows of one sequence whose queries single out one key each: itself, the first ones, those at page borders
    and far ones; and what the plain statement makes of them."""

    def __init__(self, name, T, seed=0, rising=False):
        H, dk, dv, rank, gate = self.sizes = LAT[name]
        g = torch.Generator().manual_seed(seed)
        n = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
        gw = torch.Generator().manual_seed(99)      # weights do not depend on the sequence
        nw = lambda *s: torch.randn(*s, generator=gw, dtype=torch.float64)  # noqa: E731
        self.w_norm = r16(1 + 0.2 * nw(rank))
        self.uk, self.uv = r16(nw(H * dk, rank) * rank ** -0.5), r16(nw(H * dv, rank) * rank ** -0.5)
        self.scale = 1.3 * dk ** -0.5
        z, gt = r16(2 * n(T, rank)), r16(n(T, H * dv))
        if rising:          # scores that keep growing along the sequence
            base = n(rank)
            z = r16(base[None] * (torch.arange(T)[:, None] / T) + 0.3 * n(T, rank))
        self.c = O.rms(GAIN * z, EPS) * self.w_norm
        k = (self.c @ self.uk.T).view(T, H, dk)
        q = n(T, H, dk)
        for i in range(T):
            spots = [i, 0, 63, 64, i - 1, i // 64 * 64, i // 64 * 64 - 1, i - 128, i // 2]
            j = T - 1 if rising else spots[i % len(spots)]
            if rising or 0 <= j <= i:
                q[i] = k[j] * (14.0 / (self.scale * GAIN * (k[j] * k[j]).sum(-1, keepdim=True)))
        q = r16(q)
        o = O.latent_attention(GAIN * q, self.c, self.uk, self.uv, self.scale).reshape(T, -1)
        self.want = o * O.sigmoid(GAIN * gt) if gate else o
        up = lambda m: (m + 7) // 8 * 8  # noqa: E731
        qo = 8
        co = qo + up(H * dk)
        go = co + up(rank)
        self.spec = LatentSpec(H, dk, dv, rank, qo, co, go if gate else -1, self.scale, EPS)
        x = torch.full((T, go + up(H * dv) + 8), 5.0, dtype=torch.float64)
        for off, t in ((qo, q), (co, z), (go, gt)):
            x[:, off:off + t[0].numel()] = t.reshape(T, -1)
        self.x = x

    def weights(self, dtype, device):
        to = lambda t: t.to(dtype).to(device)  # noqa: E731
        return {"c_norm": to(self.w_norm), "kv_up": to(torch.cat([self.uk, self.uv])).contiguous(),
                "gain": to(torch.tensor(GAIN))}


class Pages:
    """A cache with scattered blocks that hold what earlier sequences left."""

    def __init__(self, spec, slots, max_len, dtype, device, seed=3):
        g = torch.Generator().manual_seed(seed)
        nb = (max_len + 63) // 64
        self.table = torch.randperm(slots * nb + 3, generator=g)[: slots * nb].to(torch.int32).view(slots, nb).to(device)
        self.cache = (torch.randn(slots * nb + 3, spec.block_elems, generator=g) * 30).to(dtype).to(device)


def run_portions(case, x, w, pages, slot, cuts, out, at=0, **kw):
    for n in cuts:
        dev = x.device
        pos = torch.arange(at, at + n, dtype=torch.int32, device=dev)
        ids = torch.full((n,), slot, dtype=torch.int32, device=dev)
        latent_attention(case.spec, x[at:at + n], w, ids, pos, pages.table, pages.cache, out[at:at + n], 16,
                         plan=LatentPlan([n], [at], [slot], dev), **kw)
        at += n


def run_single(case, x, w, pages, slot, at, out):
    """One decode row in a batch with idle slots."""
    S, dev = pages.table.shape[0], x.device
    rows = torch.zeros(S, x.shape[1], dtype=x.dtype, device=dev)
    rows[slot] = x[at]
    ids = torch.full((S,), -1, dtype=torch.int32, device=dev)
    ids[slot] = slot
    pos = torch.full((S,), -1, dtype=torch.int32, device=dev)
    pos[slot] = at
    o = torch.full((S, out.shape[1]), 5.0, dtype=x.dtype, device=dev)
    latent_attention(case.spec, rows, w, ids, pos, pages.table, pages.cache, o, 16)
    out[at] = o[slot]
    idle = [s for s in range(S) if s != slot]
    assert o[idle, 16:16 + case.spec.heads * case.spec.vdim].abs().max().item() == 0


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(LAT))
def test_latent_attention_prompts_portions_and_single_tokens(name, device, dtype):
    T = 203
    case = Case(name, T)
    x, w = case.x.to(dtype).to(device), case.weights(dtype, device)
    hv = case.want.shape[1]
    fresh = lambda: torch.full((T, 16 + (hv + 7) // 8 * 8), 9.0, dtype=dtype, device=device)  # noqa: E731
    for cuts in ([T], [2, 62, 64, 1, 66, 8], [128, 75], [17, 2, 2, 2, 180]):
        pages, out = Pages(case.spec, 3, 256, dtype, device), fresh()
        run_portions(case, x, w, pages, 1, cuts, out)
        finish(device)
        close(out[:, 16:16 + hv], case.want, dtype, f"portions {cuts}")
        assert (out[:, :16] == 9).all()
    pages, out = Pages(case.spec, 3, 256, dtype, device), fresh()
    run_portions(case, x, w, pages, 2, [1], out)
    start = 97
    run_portions(case, x, w, pages, 2, [start - 1], out, at=1)
    for at in range(start, T):
        run_single(case, x, w, pages, 2, at, out)
    finish(device)
    close(out[:, 16:16 + hv], case.want, dtype, "single tokens")


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_general_kernels_take_bf16_too(name):
    case = Case(name, 130)
    x, w = case.x.bfloat16().cuda(), case.weights(torch.bfloat16, "cuda")
    pages = Pages(case.spec, 2, 192, torch.bfloat16, "cuda")
    out = torch.zeros(130, 16 + case.want.shape[1], dtype=torch.bfloat16, device="cuda")
    run_portions(case, x, w, pages, 1, [100, 30], out, simt=True)
    finish("cuda")
    close(out[:, 16:], case.want, torch.bfloat16)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name,rising", [("mixed", False), ("wide", False), ("wide", True), ("two_groups", True)])
def test_single_tokens_of_unequal_contexts_in_one_batch(name, rising, device, dtype):
    """Contexts from one token to many pages, idle rows between them: the list of tiles is cut at arbitrary places.
    ``rising``: scores that grow along the sequence, so the running maximum is raised over and over."""
    ctx = [1, 0, 64, 65, 1500 if device == "cuda" else 200, 700 if device == "cuda" else 130, 0, 63, 0]
    S = len(ctx)
    cases = [Case(name, max(n, 1), seed=i, rising=rising) for i, n in enumerate(ctx)]
    c0 = cases[0]
    w = c0.weights(dtype, device)
    pages = Pages(c0.spec, S, max(ctx), dtype, device)
    hv = c0.want.shape[1]
    rows = torch.zeros(S, c0.x.shape[1], dtype=dtype, device=device)
    for i, (c, n) in enumerate(zip(cases, ctx)):
        if n > 1:
            run_portions(c, c.x.to(dtype).to(device), w, pages, i, [n - 1],
                         torch.zeros(n, 16 + hv, dtype=dtype, device=device))
        if n:
            rows[i] = c.x[n - 1].to(dtype)
    ids = torch.tensor([i if n else -1 for i, n in enumerate(ctx)], dtype=torch.int32, device=device)
    pos = torch.tensor([n - 1 for n in ctx], dtype=torch.int32, device=device)
    out = torch.full((S, 16 + hv), 7.0, dtype=dtype, device=device)
    for _ in range(2):      # again: nothing is left over in the workspaces
        latent_attention(c0.spec, rows, w, ids, pos, pages.table, pages.cache, out, 16)
    finish(device)
    for i, (c, n) in enumerate(zip(cases, ctx)):
        if n:
            close(out[i, 16:], c.want[n - 1], dtype, f"row {i}")
        else:
            assert out[i, 16:].abs().max().item() == 0


@pytest.mark.parametrize("device,dtype", WHERE)
def test_portions_of_unequal_sequences_in_one_batch(device, dtype):
    lens, starts, slots = [1, 130, 64, 7, 40], [0, 65, 2, 70, 0], [3, 2, 1, 0, 4]
    cases = [Case("three_chunks", st + n, seed=i) for i, (n, st) in enumerate(zip(lens, starts))]
    w, hv = cases[0].weights(dtype, device), cases[0].want.shape[1]
    pages = Pages(cases[0].spec, 5, 256, dtype, device)
    for c, st, slot in zip(cases, starts, slots):
        if st:
            run_portions(c, c.x[:st].to(dtype).to(device), w, pages, slot, [st],
                         torch.zeros(st, 16 + hv, dtype=dtype, device=device))
    x = torch.cat([c.x[st:] for c, st in zip(cases, starts)]).to(dtype).to(device)
    ids = torch.cat([torch.full((n,), s, dtype=torch.int32) for n, s in zip(lens, slots)]).to(device)
    pos = torch.cat([torch.arange(st, st + n, dtype=torch.int32) for st, n in zip(starts, lens)]).to(device)
    out = torch.zeros(x.shape[0], 16 + hv, dtype=dtype, device=device)
    latent_attention(cases[0].spec, x, w, ids, pos, pages.table, pages.cache, out, 16,
                     plan=LatentPlan(lens, starts, slots, torch.device(device)))
    finish(device)
    close(out[:, 16:], torch.cat([c.want[st:] for c, st in zip(cases, starts)]), dtype)


@pytest.mark.gpu
def test_more_rows_than_one_launch_takes():
    S, ctx = 1300, 70
    case = Case("one", ctx)
    w, dev = case.weights(torch.bfloat16, "cuda"), torch.device("cuda")
    x = case.x.bfloat16().to(dev)
    pages = Pages(case.spec, S, 128, torch.bfloat16, "cuda")
    out = torch.zeros(S * 2, 16 + case.want.shape[1], dtype=torch.bfloat16, device=dev)
    for at in range(0, S, 325):
        slots = list(range(at, at + 325))
        ids = torch.repeat_interleave(torch.tensor(slots, dtype=torch.int32), ctx - 1).to(dev)
        pos = torch.arange(ctx - 1, dtype=torch.int32).repeat(325).to(dev)
        scratch = torch.zeros(325 * (ctx - 1), out.shape[1], dtype=torch.bfloat16, device=dev)
        latent_attention(case.spec, x[:ctx - 1].repeat(325, 1), w, ids, pos, pages.table, pages.cache, scratch, 16,
                         plan=LatentPlan([ctx - 1] * 325, [0] * 325, slots, dev))
    ids = torch.arange(S, dtype=torch.int32, device=dev)
    pos = torch.full((S,), ctx - 1, dtype=torch.int32, device=dev)
    latent_attention(case.spec, x[-1:].repeat(S, 1), w, ids, pos, pages.table, pages.cache, out[:S], 16)
    finish("cuda")
    close(out[:S, 16:], case.want[-1:].expand(S, -1), torch.bfloat16)


def test_the_attention_cases_show_every_key():
    """A query that loses its singled-out key, or sees one key too many or too few, is far from right."""
    case = Case("mixed", 203)
    H, dk, dv, rank, _ = case.sizes
    q = case.x[:, 8:8 + H * dk].view(-1, H, dk) * GAIN
    right = O.latent_attention(q, case.c, case.uk, case.uv, case.scale)
    for i in (9 * 14, 9 * 14 + 1, 9 * 14 + 2, 9 * 14 + 3, 9 * 14 + 5, 9 * 14 + 6, 9 * 14 + 7):
        for lose in (i, 0, 63, 64, i // 64 * 64, i // 64 * 64 - 1, i - 128):
            if [i, 0, 63, 64, i - 1, i // 64 * 64, i // 64 * 64 - 1, i - 128, i // 2][i % 9] != lose or lose < 0:
                continue
            keep = torch.tensor([j for j in range(i + 1) if j != lose])
            wrong = O.latent_attention(q[i:i + 1], case.c[keep], case.uk, case.uv, case.scale, start=i)
            assert (wrong[0] - right[i]).abs().max() > 0.3 * right[i].abs().max()
    slow = torch.zeros_like(right[150])
    for h in range(H):      # the statement itself, key by key
        s = torch.stack([(q[150, h] * (case.uk[h * dk:(h + 1) * dk] @ case.c[j])).sum() * case.scale for j in range(151)])
        p = torch.softmax(s, 0)
        slow[h] = sum(p[j] * (case.uv[h * dv:(h + 1) * dv] @ case.c[j]) for j in range(151))
    assert torch.allclose(slow, right[150], atol=1e-10)


@pytest.mark.parametrize("dtype", CUDA)
@pytest.mark.parametrize("T,H,m,r", [(1, 1, 8, 8), (130, 3, 24, 136), (33, 5, 200, 64), (7, 2, 13, 21), (257, 16, 128, 512)])
def test_head_product(T, H, m, r, dtype):
    g = torch.Generator().manual_seed(T)
    w = r16(torch.randn(H, m, r, generator=g, dtype=torch.float64) * r ** -0.5)
    simt = m % 8 != 0 or r % 8 != 0
    put = lambda t: t.to(dtype).cuda()  # noqa: E731
    gain = torch.tensor(-1.5)
    for by_rows in (True, False):
        k, n = (m, r) if by_rows else (r, m)
        pad = (H * k + 7) // 8 * 8
        a = r16(torch.randn(T, pad + 8, generator=g, dtype=torch.float64))
        gate = r16(torch.randn(T, H * n, generator=g, dtype=torch.float64))
        want = torch.einsum("thk,hkn->thn" if by_rows else "thk,hnk->thn", a[:, 8:8 + H * k].view(T, H, k), w)
        for gated in (False, True):
            out = torch.full((T, H * n), 3.0, dtype=dtype, device="cuda")
            head_product(put(a)[:, 8:], k, put(w).view(H * m, r), H, out, by_rows=by_rows, simt=simt,
                         gate=put(gate) if gated else None, gain=put(gain) if gated else None)
            ref = want.reshape(T, -1) * (O.sigmoid(gain.double() * gate) if gated else 1.0)
            close(out, ref, dtype, f"by_rows {by_rows} gated {gated}", rel=None if dtype == torch.float32 else 8e-3)
    finish("cuda")


# ---- rows ------------------------------------------------------------------------------------------------------------------
def close_rows(got, want, dtype, what=""):
    close(got, want, dtype, what, rel=2e-6 if dtype == torch.float32 else 6e-3)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,W", [(3, 64), (17, 1000), (2, 1030), (5, 51), (4, 3584), (2, 4352)])
def test_stream_update(T, W, device, dtype):
    g = torch.Generator().manual_seed(W)
    n = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    put = lambda t: t.to(dtype).to(device)  # noqa: E731
    h0 = n(T, W).float().double()
    wide = r16(n(T, 2 * W + 24))
    b1, b2, g1, g2, wt = r16(n(W)), r16(n(W)), torch.tensor(1.25), torch.tensor(-0.5), torch.tensor(1.75)
    y1, y2 = n(3, T, W).float().double(), r16(n(1, T, W))
    mult, eps = 0.3, 1e-2
    off = 16 if W % 8 == 0 else 5
    gates = put(wide)
    sub1 = R.Sublayer(y1.float().to(device), gates[:, 8:8 + W], put(b1), put(g1))
    sub2 = R.Sublayer(put(y2), gates[:, off + W - 8 if W % 8 == 0 else off + W:][:, :W], put(b2), put(g2))
    o2 = off + W - 8 if W % 8 == 0 else off + W
    add1 = y1.sum(0) * O.sigmoid(g1.double() * wide[:, 8:8 + W] + b1)
    add2 = y2[0] * O.sigmoid(g2.double() * wide[:, o2:o2 + W] + b2)
    for subs, add in (([], 0), ([sub1], add1), ([sub1, sub2], add1 + add2), ([R.Sublayer(put(y2))], y2[0])):
        h = h0.float().to(device)
        x = R.stream_update(h, subs, mult, dtype, eps)
        want = h0 + mult * add
        close(h, want, torch.float32, "stream", rel=2e-6)
        close_rows(x, O.rms(want, eps), dtype)
        h = h0.float().to(device)
        close_rows(R.stream_update(h, subs, mult, dtype, eps, weight=put(wt)), O.rms(want, eps) * 1.75, dtype)
        h = h0.float().to(device)
        parts = R.stream_update(h, subs, mult, dtype, eps, split=True)
        close(h, want, torch.float32, "stream", rel=2e-6)
        assert parts.shape[0] == (T if dtype == torch.float32 else 2 * T)
        close(parts.double().view(-1, T, W).sum(0), want, torch.float32, "two rows", rel=2e-5)
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("T,W", [(3, 64), (300, 128), (2, 51), (40, 2056)])
def test_entry_of_a_pass(T, W, device, dtype):
    """Split of the stream, both halves of the entry matrix, the vector of the pass: the stream's own 32 bits enter."""
    g = torch.Generator().manual_seed(W)
    n = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    h0, x0, w_in, step = (n(T, W) * 20).float().double(), r16(n(T, W)), r16(n(W, 2 * W) * W ** -0.5), r16(n(3, W))
    put = lambda t: t.to(dtype).to(device)  # noqa: E731
    wd = put(w_in)
    base = linear_partial(put(x0), wd[:, W:], f32=True)
    for t in range(3):
        h = h0.float().to(device)
        parts = R.stream_update(h, [], 1.0, dtype, 1e-3, split=True)
        x = R.enter_pass(h, linear_partial(parts, wd[:, :W], f32=True), base, put(step)[t], 1e-3)
        want = O.enter_pass(h0, x0, w_in, step[t])
        close(h, want, torch.float32, "stream", rel=5e-5)       # far below the 4e-3 of a rounded stream
        close_rows(x, O.rms(want, 1e-3), dtype)
    finish(device)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("I", [64, 50])
def test_activations(I, device, dtype):
    g = torch.Generator().manual_seed(I)
    x = r16(torch.randn(9, 2 * I + 24, generator=g, dtype=torch.float64) * 3)
    xd, gain = x.to(dtype).to(device), torch.tensor(-1.5)
    acts = {"gelu": O.gelu_erf, "silu": lambda z: z * O.sigmoid(z),
            "gelu_tanh": lambda z: 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))}
    for name, fn in acts.items():
        for f in (None, gain):
            got = R.scaled_act(xd[:, 8:8 + I], name, f.to(dtype).to(device) if f is not None else None)
            close_rows(got, fn(x[:, 8:8 + I] * (f.double() if f is not None else 1.0)), dtype, name)
        pair = x[:, :2 * I]
        close_rows(R.gated_act(xd[:, :2 * I].contiguous(), name), fn(pair[:, :I]) * pair[:, I:], dtype, name)
    # the exact form, not the tanh one
    z = torch.linspace(-4, 4, 41, dtype=torch.float64)
    assert (acts["gelu"](z) - acts["gelu_tanh"](z)).abs().max() > 3e-4
    if dtype == torch.float32:
        got = R.scaled_act(z.float()[None].to(device), "gelu").double().cpu()[0]
        assert (got - acts["gelu"](z)).abs().max() < 2e-6
    finish(device)


@pytest.mark.parametrize("dtype", CUDA)
@pytest.mark.parametrize("M", [1, 60, 200, 600])
@pytest.mark.parametrize("N,K", [(256, 512), (72, 2048), (1536, 1536), (51, 40)])
def test_partial_products_add_up(M, N, K, dtype):
    g = torch.Generator().manual_seed(M)
    a, w = r16(torch.randn(M, K, generator=g, dtype=torch.float64)), r16(torch.randn(N, K, generator=g, dtype=torch.float64))
    for f32 in (False, True):
        y = linear_partial(a.to(dtype).cuda(), w.to(dtype).cuda(), f32)
        assert y.dim() == 3 and (y.dtype == torch.float32 or not f32)
        close(y.double().sum(0), a @ w.T, dtype, rel=4e-3 if y.dtype == torch.bfloat16 else 1e-5)
    finish("cuda")
