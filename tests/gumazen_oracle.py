"""Plain, slow statement of the Gumazen decoder in float64: one function per mechanism, whole sequences, no cache, no
batching, every expert as its own product.  It is written from the equations and imports nothing of the package, so the
tests compare two independent programs.  ``weights`` maps checkpoint names to tensors, ``cfg`` is the parsed config.json."""
from __future__ import annotations

import math

import torch


# ---- norms, activations ----------------------------------------------------------------------------------------------------
def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# ---- positions --------------------------------------------------------------------------------------------------------------
def frequencies(rot):
    """One angular frequency per rotated pair, with the three-band scaling when the config has one."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate(x, positions, rot):
    """``x [T, heads, dim]``: pairs (i, i + dims / 2) of the first ``dims`` dimensions turn by ``position * f_i``."""
    half = rot["dims"] // 2
    y = x.clone()
    for i, f in enumerate(frequencies(rot)):
        a = positions.double() * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * c - v * s
        y[..., i + half] = v * c + u * s
    return y


def bucket(n, rows, far):
    """Row of the distance table: the first half one row per distance, the rest logarithmic up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


# ---- attention -------------------------------------------------------------------------------------------------------------
def attend(q, k, v, scale, start=0, window=0, cap=0.0, bias=None, sink=False):
    """``q [Tq, H, dim]`` at positions ``start ..`` over ``k [T, G, dim]``, ``v [T, G, vdim]``; ``bias [rows of distances,
    H]`` is indexed by the distance itself."""
    Tq, H, _ = q.shape
    T, G, _ = k.shape
    out = torch.zeros(Tq, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for t in range(Tq):
            i = start + t
            lo = max(0, i - window + 1) if window else 0
            s = (k[lo:i + 1, g] @ q[t, h]) * scale
            if cap:
                s = cap * torch.tanh(s / cap)
            if bias is not None:
                s = s + bias[torch.arange(i - lo, -1, -1), h]
            top = torch.maximum(s.max(), torch.zeros(())) if sink else s.max()
            e = torch.exp(s - top)
            den = e.sum() + (torch.exp(-top) if sink else 0.0)
            out[t, h] = (e / den) @ v[lo:i + 1, g]
    return out


def mixer(kind, h, W, p, m, eps):
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    pos = torch.arange(T)

    def project(name):
        y = h @ W[p + name].T
        return y + W[p + name + ".b"] if kind == "attention_3" else y
    q, k, v = project("q"), project("k"), project("v")
    if kind in ("attention_2", "attention_3"):
        q, k = rms(q, eps) * W[p + "q.norm"], rms(k, eps) * W[p + "k.norm"]
    q, k, v = q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1)
    if kind in ("attention", "attention_3"):
        q, k = rotate(q, pos, m["rot"]), rotate(k, pos, m["rot"])
    if kind == "attention":
        o = attend(rms(q, eps), rms(k, eps), v, m["scale"], sink=True)
    elif kind == "attention_2":
        rel = W[p + "rel"]
        rows = torch.tensor([bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)])
        o = attend(q, k, v, m["scale"], window=m["mask"]["size"], cap=m["softcap"], bias=rel[rows])
        o = o * sigmoid(h @ W[p + "g"].T)[:, :, None]
    else:
        o = attend(q, k, v, m["scale"])
    y = o.reshape(T, -1) @ W[p + "o"].T
    return y + W[p + "o.b"] if kind == "attention_3" else y


# ---- feed-forward ----------------------------------------------------------------------------------------------------------
def dense(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def expert(h, W, p):
    z = h @ W[p + "gate"].T
    return (z * sigmoid(z) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, correction, r):
    """Chosen ids (experts, then identity experts) and their weights for one token's router logits ``z``."""
    e = torch.exp(z - z.max())
    s = e / e.sum()
    choice = (s + correction).tolist()
    n = r["groups"]["count"]
    size = len(choice) // n
    best = [max(choice[g * size:(g + 1) * size]) for g in range(n)]
    kept = sorted(range(n), key=lambda g: -best[g])[:r["groups"]["keep"]]
    allowed = [i for i in range(len(choice)) if i // size in kept]
    ids = sorted(allowed, key=lambda i: -choice[i])[:r["top"]]
    w = s[ids]
    return ids, w / (w.sum() + 1e-20) * r["scale"]


def mixture(h, W, p, m):
    r = m["router"]
    out = expert(h, W, p + "shared.") if m.get("shared") else torch.zeros_like(h)
    z = h @ W[p + "router"].T
    for t in range(h.shape[0]):
        for i, w in zip(*route(z[t], W[p + "correction"], r)):
            out[t] += w * (h[t] if i >= r["experts"] else expert(h[t:t + 1], W, p + f"e{i}.")[0])
    return out


def feed_forward(h, W, p, m):
    return dense(h, W, p) if m["kind"] == "dense" else mixture(h, W, p, m)


# ---- layers ----------------------------------------------------------------------------------------------------------------
def sublayer(xs, W, p, q, eps, fn):
    """Hyper-connection ``q`` of the layer around ``fn``; ``xs`` is the list of streams."""
    w_in, w_out, w_mix = W[p + f"hc{q}.in"], W[p + f"hc{q}.out"], W[p + f"hc{q}.mix"]
    n = len(xs)
    u = sum(w_in[s] * xs[s] for s in range(n))
    y = fn(layer_norm(u, W[p + f"norm{q}"], W[p + f"norm{q}.b"], eps))
    return [sum(w_mix[s, t] * xs[s] for s in range(n)) + w_out[t] * y for t in range(n)]


def layer(xs, W, p, c, eps):
    xs = sublayer(xs, W, p, 1, eps, lambda h: mixer(c["type"], h, W, p + "mix.", c["mixer"], eps))
    if c["mlp"] is not None:
        xs = sublayer(xs, W, p, 2, eps, lambda h: feed_forward(h, W, p + "mlp.", c["mlp"]))
    return xs


def run_order(cfg):
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def forward(cfg, weights, tokens, streams=None):
    """Logits ``[T, vocab]``; ``streams`` (a list) receives the sum of the streams after every layer run."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    xs = [W["embed"][torch.tensor(tokens)]] * cfg["streams"]
    for i in run_order(cfg):
        xs = layer(xs, W, f"l{i}.", cfg["layers"][i], eps)
        if streams is not None:
            streams.append(sum(xs))
    return layer_norm(sum(xs), W["final.norm"], W["final.norm.b"], eps) @ W["head"].T


# ---- random checkpoints ----------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """Names and shapes of the checkpoint of a config (``rel_rows`` of a mixer: rows of its distance table)."""
    w, s = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": (w,), "final.norm.b": (w,)}
    for i, c in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", c["mixer"], c["mlp"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for q in (1, 2) if f else (1,):
            out.update({p + f"norm{q}": (w,), p + f"norm{q}.b": (w,), p + f"hc{q}.in": (s,), p + f"hc{q}.out": (s,),
                        p + f"hc{q}.mix": (s, s)})
        out.update({p + "mix.q": (H * dk, w), p + "mix.k": (G * dk, w), p + "mix.v": (G * dv, w), p + "mix.o": (w, H * dv)})
        if c["type"] in ("attention_2", "attention_3"):
            out.update({p + "mix.q.norm": (H * dk,), p + "mix.k.norm": (G * dk,)})
        if c["type"] == "attention_2":
            out.update({p + "mix.rel": (c["rel_rows"], H), p + "mix.g": (H, w)})
        if c["type"] == "attention_3":
            out.update({p + "mix.q.b": (H * dk,), p + "mix.k.b": (G * dk,), p + "mix.v.b": (G * dv,), p + "mix.o.b": (w,)})
        if f and f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], w), p + "mlp.down": (w, f["ff"])})
        elif f:
            r = f["router"]
            n = r["experts"] + r.get("identity", 0)
            out.update({p + "mlp.router": (n, w), p + "mlp.correction": (n,)})
            for name, ff in [(f"e{e}.", f["expert"]["ff"]) for e in range(r["experts"])] + (
                    [("shared.", f["shared"]["ff"])] if f.get("shared") else []):
                out.update({p + "mlp." + name + "gate": (ff, w), p + "mlp." + name + "up": (ff, w),
                            p + "mlp." + name + "down": (w, ff)})
    return out


def random_checkpoint(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(*shape, generator=g)
        last = name.split(".")[-1]
        if name == "embed":
            pass
        elif ".hc" in name:
            t = t * 0.25 + (torch.eye(shape[0]) if last == "mix" else (1.0 / shape[0] if last == "in" else 1.0))
        elif last.startswith("norm"):
            t = 1.0 + 0.3 * t
        elif last == "b":
            t = 0.2 * t
        elif last == "rel":
            t = 1.5 * t
        elif last == "correction":
            t = 0.1 * t
        elif last == "router":
            t = t * 2.0 * shape[-1] ** -0.5
        else:
            t = t * shape[-1] ** -0.5
        W[name] = t.bfloat16()
    return W
