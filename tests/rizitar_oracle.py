"""Plain, slow statement of the Rizitar decoder in float64: one function per mechanism, whole sequences, no cache, no batching,
every expert as its own product.  It is written from the equations and imports nothing of the package, so the tests compare two
independent programs.  ``weights`` maps checkpoint names to tensors, ``cfg`` is the parsed config.json."""
from __future__ import annotations

import math

import torch


# ---- norms, activations ----------------------------------------------------------------------------------------------------
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def xielu(z, p, q):
    """Quadratic with slope one half on the right, exponential with the same slope at zero on the left."""
    right = softplus(p) * z * z + 0.5 * z
    low = torch.clamp(z, max=0.0)
    left = (0.5 + softplus(q)) * (torch.expm1(low) - low) + 0.5 * z
    return torch.where(z > 0, right, left)


# ---- positions --------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """One angular frequency per rotated pair and the factor of cosines and sines (YaRN when the config has a scaling)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def dim_of(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / sc["factor"] * r + x * (1.0 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """``x [T, heads, dim]``: pairs (i, i + dims / 2) of the first ``dims`` dimensions turn by ``position * f_i``."""
    half = rot["dims"] // 2
    freq, mag = frequencies(rot)
    y = x.clone()
    for i, f in enumerate(freq):
        a = positions.double() * f
        c, s = (mag * torch.cos(a))[:, None], (mag * torch.sin(a))[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i], y[..., i + half] = u * c - v * s, v * c + u * s
    return y


# ---- attention --------------------------------------------------------------------------------------------------------------
def pooled(x, pool):
    """Means of the whole blocks of ``pool`` rows: ``x [T, heads, dim]`` -> ``[T // pool, heads, dim]``."""
    n = x.shape[0] // pool
    return x[:n * pool].reshape(n, pool, *x.shape[1:]).mean(1)


def window_scores(q, k, scale, window, pool):
    """Scores of one head (``q [T, d]``, ``k [T, d]``) against tokens and pooled blocks with the hidden ones at -inf:
    ``[T, T + blocks]``."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    seen = j <= i
    if window:
        seen = seen & (i - j < window)
    s = (q @ k.t() * scale).masked_fill(~seen, -math.inf)
    if window and pool:
        kb = pooled(k[:, None], pool)[:, 0]
        b = torch.arange(kb.shape[0])[None]
        s = torch.cat([s, (q @ kb.t() * scale).masked_fill((b + 1) * pool - 1 > i - window, -math.inf)], 1)
    return s


def attend(q, k, v, sink, scale, window, pool):
    """``q [T, H, d]``, ``k / v [T, G, ..]`` -> ``[T, H, dv]``; ``sink [H]`` or None."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = window_scores(q[:, h], k[:, g], scale, window, pool)
        vals = v[:, g]
        if s.shape[1] > T:
            vals = torch.cat([vals, pooled(v[:, g:g + 1], pool)[:, 0]])
        if sink is not None:
            s = torch.cat([s, sink[h].expand(T, 1)], 1)
        w = torch.softmax(s, -1)
        out.append(w[:, :vals.shape[0]] @ vals)
    return torch.stack(out, 1)


def attention(h, m, w, eps, positions):
    """``w``: tensors of the mixer by their short names."""
    T = h.shape[0]
    q = (h @ w["q"].t()).reshape(T, m["heads"], m["dim"])
    k = (h @ w["k"].t()).reshape(T, m["kv_heads"], m["dim"])
    v = k
    q, k = rms(q, eps) * w["q.norm"], rms(k, eps) * w["k.norm"]
    if m.get("rot"):
        q, k = rotate(q, positions, m["rot"]), rotate(k, positions, m["rot"])
    mask = m.get("mask") or {}
    o = attend(q, k, v, w["sink"], m["scale"], mask.get("size") or 0, mask.get("pool") or 0)
    return o.reshape(T, -1) @ w["o"].t()


# ---- generalized delta rule -------------------------------------------------------------------------------------------------
def delta_gates(h, w):
    """Decay and removal rate of every head's key channels: ``[T, heads * dim]`` each."""
    z = torch.tanh(h @ w["w1"].t()) @ w["w2"].t() + w["w0"]
    return torch.exp(-math.exp(-0.5) * sigmoid(z)), sigmoid(h @ w["a"].t() + w["a.b"])


def delta_scan(r, k, v, decay, rate, S=None):
    """``[T, H, d]`` each; one token after the other.  Returns ``o [T, H, d]`` and the last state ``[H, d, d]``."""
    T, H, d = r.shape
    S = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if S is None else S
    out = []
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum(-1, keepdim=True) + 1e-6)
        seen = torch.einsum("hk,hkv->hv", u, S)
        S = decay[t][:, :, None] * S - (rate[t] * u)[:, :, None] * seen[:, None] + k[t][:, :, None] * v[t][:, None]
        out.append(torch.einsum("hk,hkv->hv", r[t], S))
    return torch.stack(out) if T else r.new_zeros(0, H, v.shape[2]), S


def general_delta(h, m, w, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    split = lambda x: x.reshape(T, H, d)  # noqa: E731
    decay, rate = delta_gates(h, w)
    o, _ = delta_scan(split(h @ w["r"].t()), split(h @ w["k"].t()), split(h @ w["v"].t()), split(decay), split(rate))
    return (rms(o, eps).reshape(T, H * d) * w["norm"] * sigmoid(h @ w["g"].t())) @ w["o"].t()


# ---- feed-forwards, token input ---------------------------------------------------------------------------------------------
def dense(h, w):
    return xielu(h @ w["up"].t() + w["up.b"], w["act"][0], w["act"][1]) @ w["down"].t() + w["down.b"]


def route(z, top):
    """Weights and ids ``[T, top]`` of the chosen experts: the soft-max scores as they are."""
    s = torch.softmax(z, -1)
    ids = torch.sort(s, dim=-1, descending=True, stable=True).indices[:, :top]
    return s.gather(1, ids), ids


def experts(h, w, ids, ups, downs):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for x, e in zip(w[t], ids[t].tolist()):
            a = torch.clamp(ups[e] @ h[t], min=0.0) ** 2
            out[t] += x * (downs[e] @ a)
    return out


def routed(h, mlp, w):
    r = mlp["router"]
    ws, ids = route(h @ w["router"].t(), r["top"])
    return experts(h, ws, ids, [w[f"e{j}.up"] for j in range(r["experts"])], [w[f"e{j}.down"] for j in range(r["experts"])])


def token_side(x, e, w, eps):
    """What the layer's own token vectors ``e [T, dim]`` add to the stream ``x``."""
    return rms((gelu_tanh(x @ w["gate"].t()) * e) @ w["proj"].t(), eps) * w["norm"]


# ---- the model --------------------------------------------------------------------------------------------------------------
def _part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence."""
    weights = {k: v.double() for k, v in weights.items()}
    tok = torch.as_tensor(tokens)
    positions = torch.arange(len(tok))
    eps = cfg["norm"]["eps"]
    x = weights["embed"][tok] * cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * weights[p + "norm1"]
        mix = _part(weights, p + "mix.")
        y = attention(h, lay["mixer"], mix, eps, positions) if lay["type"] == "attention" else \
            general_delta(h, lay["mixer"], mix, eps)
        x = x + rms(y, eps) * weights[p + "norm1b"]
        if lay.get("mlp"):
            h = rms(x, eps) * weights[p + "norm2"]
            y = dense(h, _part(weights, p + "mlp.")) if lay["mlp"]["kind"] == "dense" else \
                routed(h, lay["mlp"], _part(weights, p + "mlp."))
            x = x + rms(y, eps) * weights[p + "norm2b"]
        n = cfg["token_side"]["dim"]
        x = x + token_side(x, weights["side.embed"][tok][:, i * n:(i + 1) * n], _part(weights, p + "side."), eps)
        if layers_out is not None:
            layers_out.append(x)
    return rms(x, eps) * weights["final.norm"] @ weights["embed"].t()


# ---- random checkpoints ----------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """Names and shapes of the checkpoint of a config (``rank`` of a layer: low-rank width of its decay)."""
    w, n = cfg["width"], cfg["token_side"]["dim"]
    out = {"embed": (cfg["vocab"], w), "side.embed": (cfg["vocab"], n * len(cfg["layers"])), "final.norm": (w,)}
    for i, c in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", c["mixer"], c["mlp"]
        out.update({p + k: (w,) for k in (("norm1", "norm1b", "norm2", "norm2b") if f else ("norm1", "norm1b"))})
        out.update({p + "side.gate": (n, w), p + "side.proj": (w, n), p + "side.norm": (w,)})
        hd = m["heads"] * m["dim"]
        out[p + "mix.o"] = (w, hd)
        if c["type"] == "attention":
            out.update({p + "mix.q": (hd, w), p + "mix.k": (m["kv_heads"] * m["dim"], w), p + "mix.q.norm": (m["dim"],),
                        p + "mix.k.norm": (m["dim"],), p + "mix.sink": (m["heads"],)})
        else:
            out.update({p + "mix." + k: (hd, w) for k in ("r", "k", "v", "g", "a")})
            out.update({p + "mix.a.b": (hd,), p + "mix.w0": (hd,), p + "mix.norm": (hd,), p + "mix.w1": (c["rank"], w),
                        p + "mix.w2": (hd, c["rank"])})
        if f and f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], w), p + "mlp.up.b": (f["ff"],), p + "mlp.down": (w, f["ff"]),
                        p + "mlp.down.b": (w,), p + "mlp.act": (2,)})
        elif f:
            out[p + "mlp.router"] = (f["router"]["experts"], w)
            for e in range(f["router"]["experts"]):
                out.update({p + f"mlp.e{e}.up": (f["expert"]["ff"], w), p + f"mlp.e{e}.down": (w, f["expert"]["ff"])})
    return out


def random_checkpoint(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        last = name.split(".")[-1]
        if last.startswith("norm"):
            t = 1.0 + 0.3 * t
        elif last == "sink":
            t = 1.5 + t
        elif last in ("b", "w0"):
            pass
        elif name == "embed":
            t = 1.5 * t * shape[-1] ** -0.5
        elif last == "embed":
            t = 1.5 * t
        elif last == "act":
            t = 0.7 * t
        elif last == "router":
            t = t * 2.0 * shape[-1] ** -0.5
        elif len(shape) > 1:
            t = t * shape[-1] ** -0.5
        W[name] = t.bfloat16()
    return W
