"""Serving throughput of a hybrid decoder (Domavik, Poralorn, Gumazen, Rizitar) beside the closest decoder of equal size, and its kernels
beside the like kernels of that model.

    python bench.py --workload serve [--design poralorn|gumazen|rizitar]             # end to end, a few sizes
    python -m siirl_b200.benchmarks.hybrid_serving [--design poralorn|gumazen|rizitar] --kernels

End to end: random weights, the rollout engine's own prefill pass and CUDA-graph decode rounds, CUDA events on the
launching stream.  Weights and caches are larger than L2 in every case.  Kernels: each alone as a CUDA graph, L2 flushed between
iterations, against the measured copy bandwidth and GEMM rate (MEASURED_PEAKS.json, else the figures below)."""
from __future__ import annotations

import argparse
import copy
import json
import os
from typing import Callable, Dict, List

import torch

from ..engine.rollout.native_engine import RolloutEngine, SamplingParams, _Seq
from ..models.config import DecoderConfig, get_config
from ..models.decoder import build_model
from ..ops import lib

SIZES = {     # design -> size: preset, layers, (prompts, tokens) of a prefill pass, (sequences, context) of a decode step
    "domavik": {"1.5b": ("domavik-1.5b", 14, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)]),
                "7b": ("domavik-7b", 8, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)])},
    "poralorn": {"1.5b": ("poralorn-1.5b", 14, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)]),
                 "7b": ("poralorn-7b", 8, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)])},
    "gumazen": {"a1b": ("gumazen-a1b", 12, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)]),
                "a3b": ("gumazen-a3b", 12, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)])},
    "rizitar": {"a1b": ("rizitar-a1b", 18, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)]),
                "a3b": ("rizitar-a3b", 18, [(8, 1024), (1, 8192)], [(32, 2048), (256, 1024)])},
}


def peaks() -> Dict[str, float]:
    here = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(here, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return {"gbs": p["hbm_gbs"], "tflops": p["bf16_tflops"], "source": "measured"}
    except (OSError, KeyError, ValueError):
        return {"gbs": 6650.0, "tflops": 1590.0, "source": "fallback"}


def closest(cfg: DecoderConfig) -> DecoderConfig:
    """The uniform decoder of the same width, feed-forward, number of layer runs, vocabulary and attention heads (seven
    query heads, or six, per key-value head where the design shares one latent between all); with experts where the design
    has them: as many, as many per token, as wide (two thirds where the design's experts have no gate: equal parameters), and
    a shared one."""
    b = cfg.hybrid.attention[0]
    kv = b.kv_heads or b.heads // (7 if b.heads % 7 == 0 else 6)
    moe = next((x.moe for x in cfg.hybrid.layers if x.moe is not None), None)
    if moe is not None:
        wide = moe.ff if moe.gated else moe.ff * 2 // 3
        return DecoderConfig(model_type="qwen2_moe", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size,
                             intermediate_size=cfg.intermediate_size * 2 // 3 // 64 * 64, num_layers=len(cfg.hybrid.runs()),
                             num_heads=b.heads, num_kv_heads=kv, head_dim=b.dim, rope_theta=1e6, eos_token_id=2,
                             num_experts=moe.experts, num_experts_per_tok=moe.top, moe_intermediate_size=wide,
                             tie_word_embeddings=cfg.tie_word_embeddings,
                             shared_expert_intermediate_size=moe.shared_ff, first_k_dense_replace=1)
    return DecoderConfig(model_type="qwen2", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size,
                         intermediate_size=cfg.intermediate_size, num_layers=len(cfg.hybrid.runs()), num_heads=b.heads,
                         num_kv_heads=kv, head_dim=b.dim, rope_theta=1e6, eos_token_id=2)


def closest_latent(cfg: DecoderConfig) -> DecoderConfig:
    """The dense multi-head-latent-attention decoder of the same sizes (with a 64-wide rotary part)."""
    b = cfg.hybrid.attention[0]
    n = len(cfg.hybrid.runs())
    return DecoderConfig(model_type="deepseek_v3", vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size,
                         intermediate_size=cfg.intermediate_size, num_layers=n, num_heads=b.heads, num_kv_heads=b.heads,
                         head_dim=b.dim + 64, qkv_bias=False, kv_lora_rank=b.kv_rank, qk_nope_head_dim=b.dim,
                         qk_rope_head_dim=64, v_head_dim=b.vdim, first_k_dense_replace=n, eos_token_id=2)


def _events(fn: Callable[[], None], warmup: int, iters: int, flush=None) -> float:
    """Median milliseconds of ``fn`` on the current stream."""
    times: List[float] = []
    for i in range(warmup + iters):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        if i >= warmup:
            times.append(a.elapsed_time(b))
    return sorted(times)[len(times) // 2]


def serve_one(cfg: DecoderConfig, prefill, decode, iters: int) -> dict:
    model = build_model(cfg, dtype=torch.bfloat16, device="cuda", seed=0)
    for p in model.parameters():
        p.requires_grad_(False)
    out = {"parameters": cfg.num_parameters(), "prefill": [], "decode": []}
    g = torch.Generator().manual_seed(0)
    for n, length in prefill:
        eng = RolloutEngine(model, max_num_seqs=n, max_model_len=length + 64,
                            num_blocks=n * ((length + 63) // 64 + 1), use_cuda_graph=False)
        eng._ensure_slots(n)
        eng._reset_slots()
        toks = [torch.randint(3, cfg.vocab_size, (length,), generator=g).tolist() for _ in range(n)]
        seqs = [_Seq(i, 0, length, 0, slot=i) for i in range(n)]
        for s in seqs:
            s.blocks = [eng.alloc.alloc() for _ in range((length + 63) // 64)]
        eng._write_block_tables(seqs)
        ms = _events(lambda: eng._prefill(seqs, toks), 3, iters)
        out["prefill"].append({"prompts": n, "tokens": length, "ms": round(ms, 3),
                               "tokens_per_s": round(n * length / ms * 1e3)})
        eng.sleep()
    for n, ctx in decode:
        steps = 8
        eng = RolloutEngine(model, max_num_seqs=n, max_model_len=ctx + 8 * steps + 64,
                            num_blocks=n * ((ctx + 8 * steps + 127) // 64), sync_interval=steps,
                            max_num_batched_tokens=max(ctx * n, 8192))
        times: List[float] = []
        run = eng._run_decode_steps

        def timed(k, *a, **kw):
            x, y = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            x.record()
            run(k, *a, **kw)
            y.record()
            torch.cuda.synchronize()
            times.append(x.elapsed_time(y) / k)
        eng._run_decode_steps = timed
        prompt = torch.randint(3, cfg.vocab_size, (ctx,), generator=g).tolist()
        eng.max_num_batched_tokens = 8192
        eng.generate([prompt[i:] + prompt[:i] for i in range(n)],
                     SamplingParams(n=1, temperature=1.0, max_new_tokens=1 + 6 * steps, ignore_eos=True))
        full = times[-5:-1]      # every sequence active, graph captured
        ms = sorted(full)[len(full) // 2]
        out["decode"].append({"sequences": n, "context": ctx, "ms_per_step": round(ms, 4),
                              "tokens_per_s": round(n / ms * 1e3)})
        eng.sleep()
    lib.check_status()
    del model
    torch.cuda.empty_cache()
    return out


def serve_latent(cfg: DecoderConfig, prefill, decode, iters: int) -> dict:
    """The same measurements through the latent-cache engine."""
    from ..engine.rollout.latent_engine import LatentCacheEngine
    model = build_model(cfg, dtype=torch.bfloat16, device="cuda", seed=0)
    for p in model.parameters():
        p.requires_grad_(False)
    out = {"parameters": cfg.num_parameters(), "prefill": [], "decode": []}
    g = torch.Generator().manual_seed(0)
    for n, length in prefill:
        eng = LatentCacheEngine(model, max_num_seqs=n, max_model_len=length + 64)
        eng.wake_up()
        toks = [torch.randint(3, cfg.vocab_size, (length,), generator=g).tolist() for _ in range(n)]
        ms = _events(lambda: eng._prefill(toks, list(range(n)), None), 3, iters)
        out["prefill"].append({"prompts": n, "tokens": length, "ms": round(ms, 3),
                               "tokens_per_s": round(n * length / ms * 1e3)})
        eng.sleep()
    for n, ctx in decode:
        eng = LatentCacheEngine(model, max_num_seqs=n, max_model_len=ctx + 64)
        eng.wake_up()
        tok = torch.randint(3, cfg.vocab_size, (n,), generator=g).cuda()
        slots, lens = torch.arange(n, device="cuda"), torch.full((n,), ctx, dtype=torch.int64, device="cuda")
        ms = _events(lambda: eng._logits(eng._decode(tok, slots, lens, ctx, True)), 3, iters)
        out["decode"].append({"sequences": n, "context": ctx, "ms_per_step": round(ms, 4),
                              "tokens_per_s": round(n / ms * 1e3)})
        eng.sleep()
    lib.check_status()
    del model
    torch.cuda.empty_cache()
    return out


def serve(design: str = "domavik", sizes=None, iters: int = 5) -> dict:
    res = {"metric": "serving_tokens_per_second", "data": "synthetic", "dtype": "bf16", "sizes": {}}
    for name in sizes or SIZES[design]:
        preset, layers, prefill, decode = SIZES[design][name]
        cfg = copy.deepcopy(get_config(preset))
        cfg.hybrid.layers = cfg.hybrid.layers[:layers]
        cfg.num_layers = layers
        res["sizes"][name] = {"hybrid": preset, "layers": layers, "layer_runs": len(cfg.hybrid.runs()),
                              design: serve_one(cfg, prefill, decode, iters),
                              "closest (uniform attention)": serve_one(closest(cfg), prefill, decode, iters)}
        if design == "poralorn":
            res["sizes"][name]["closest (multi-head latent attention)"] = serve_latent(closest_latent(cfg), prefill, decode,
                                                                                       iters)
    return res


# ---- kernels ----------------------------------------------------------------------------------------------------------------
class _Bench:
    def __init__(self, only: str, iters: int):
        self.only, self.iters, self.pk, self.rows = only, iters, peaks(), []
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")

    def add(self, name, fn, flops=0.0, nbytes=0.0):
        if self.only and self.only not in name:
            return
        ms = _events(self.captured(fn), 3, self.iters, self.flush)
        ideal = max(flops / (self.pk["tflops"] * 1e9), nbytes / (self.pk["gbs"] * 1e6))
        self.rows.append({"kernel": name, "us": round(ms * 1e3, 1), "roofline_us": round(ideal * 1e3, 1),
                          "of_roofline": round(ideal / ms, 3)})

    @staticmethod
    def captured(fn):
        """The launches of ``fn`` as a CUDA graph: what the host does between them (tens of microseconds) is left out."""
        side = torch.cuda.Stream()
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            fn()
        torch.cuda.current_stream().wait_stream(side)
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph):
            fn()
        return graph.replay

    def result(self):
        torch.cuda.synchronize()
        lib.check_status()
        return {"peaks": self.pk, "kernels": self.rows}


def _rnd(*s):
    return (torch.randn(*s, device="cuda") * 0.5).bfloat16()


def kernels(design: str = "domavik", only: str = "", iters: int = 20) -> dict:
    b = _Bench(only, iters)
    {"poralorn": _kernels_poralorn, "gumazen": _kernels_gumazen, "rizitar": _kernels_rizitar,
     "domavik": _kernels_domavik}[design](b)
    return b.result()


def _kernels_poralorn(b: _Bench) -> None:
    """Latent attention with 28 heads of width 128 over 512-wide latents, and the row operations of its layers."""
    from ..ops import dense, kv_cache
    from ..ops import latent_attention as LA
    from ..ops import rows as R
    from ..ops.attention import SeqInfo, attention_packed
    dev, add, rnd = torch.device("cuda"), b.add, _rnd
    H, G, D, rank = 28, 4, 128, 512
    hd = H * D
    spec = LA.LatentSpec(H, D, D, rank, 0, hd, hd + rank, D ** -0.5, 1e-5)
    w = {"c_norm": rnd(rank), "kv_up": rnd(2 * hd, rank) * 0.1, "gain": torch.ones((), device=dev).bfloat16()}
    width = 2 * hd + rank
    for n, L in ((8, 1024), (1, 8192)):
        T, nb = n * L, L // 64
        x, q = rnd(T, width), rnd(T, (H + 2 * G) * D)
        info = SeqInfo([L] * n, device=dev)
        flops = n * 4 * D * H * L * (L + 1) / 2
        table = torch.randperm(n * nb, device=dev).to(torch.int32).view(n, nb)
        cache = torch.zeros(n * nb, 64 * rank, dtype=torch.bfloat16, device=dev)
        out = torch.empty(T, hd, dtype=torch.bfloat16, device=dev)
        ids = torch.repeat_interleave(torch.arange(n, dtype=torch.int32), L).to(dev)
        pos = torch.arange(L, dtype=torch.int32).repeat(n).to(dev)
        plan = LA.LatentPlan([L] * n, [0] * n, list(range(n)), dev)
        kv = dense.linear(rnd(T, rank), w["kv_up"])
        add(f"uniform: fmha_fwd {n}x{L}", lambda: attention_packed(q, info, H, G, D), flops)
        add(f"poralorn: attention over expanded keys, gated {n}x{L}",
            lambda: LA.expanded_attention(spec, x, w["gain"], kv, ids, pos, table, out, 0, plan), flops,
            nbytes=T * hd * 10)
        add(f"poralorn: latent append {n}x{L}", lambda: LA.latent_append(spec, x, w, ids, pos, table, cache, plan),
            nbytes=T * rank * 6)
        add(f"poralorn: whole latent attention {n}x{L} (append, expansion, attention)",
            lambda: LA.latent_attention(spec, x, w, ids, pos, table, cache, out, 0, plan=plan),
            flops + T * 4.0 * hd * rank)
    for B, ctx in ((32, 2048), (256, 1024)):
        nb = (ctx + 63) // 64
        table = torch.randperm(B * nb, device=dev).to(torch.int32).view(B, nb)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, kvc = rnd(B, (H + 2 * G) * D), torch.zeros(B * nb, 2, G, 64, D, dtype=torch.bfloat16, device=dev)
        add(f"uniform: decode attention {B}x{ctx}", lambda: kv_cache.decode_attention(q, kvc, lens, table, H, G, D),
            nbytes=B * ctx * 2 * G * D * 2)
        cache = (torch.randn(B * nb, 64 * rank, device=dev) * 0.1).bfloat16()
        x, out = rnd(B, width), torch.empty(B, hd, dtype=torch.bfloat16, device=dev)
        ids, pos = torch.arange(B, dtype=torch.int32, device=dev), lens - 1
        qa, mixed = rnd(B, H * rank), torch.empty(B, H * rank, dtype=torch.bfloat16, device=dev)
        act = B * H * (D + rank) * 2
        add(f"poralorn: absorbed attention {B}x{ctx}",
            lambda: LA.absorbed_attention(spec, x, w, qa, ids, pos, table, cache, mixed),
            nbytes=B * ctx * rank * 2 + 2 * B * H * rank * 2, flops=B * ctx * H * rank * 4.0)
        add(f"poralorn: query absorption {B}", lambda: LA.head_product(x, D, w["kv_up"][:hd], H, qa, by_rows=True),
            nbytes=hd * rank * 2 + act)
        add(f"poralorn: value expansion, gated {B}",
            lambda: LA.head_product(mixed, rank, w["kv_up"][hd:], H, out, by_rows=False, gate=x[:, hd + rank:],
                                    gain=w["gain"]), nbytes=hd * rank * 2 + act + B * hd * 2)
        add(f"poralorn: whole latent attention {B}x{ctx} (append, absorption, attention, expansion)",
            lambda: LA.latent_attention(spec, x, w, ids, pos, table, cache, out, 0),
            nbytes=B * ctx * rank * 2 + 2 * hd * rank * 2 + 2 * act, flops=B * ctx * H * rank * 4.0)
    for T in (256, 8192):
        W, I = 3584, 18944
        h, p = torch.randn(T, W, device=dev), rnd(T, 2 * W)
        bias, one, step = rnd(W), w["gain"], rnd(W)
        d, res, wt = rnd(T, W), rnd(T, W), rnd(W)
        add(f"uniform: residual + RMS norm {T}x{W} (bf16 stream)", lambda: dense.rmsnorm(d, wt, 1e-6, residual=res),
            nbytes=T * W * 8)
        subs = [R.Sublayer(rnd(1, T, W), p[:, :W], bias, one), R.Sublayer(rnd(1, T, W), p[:, W:], bias, one)]
        add(f"poralorn: gated residual + norm {T}x{W} (fp32 stream)",
            lambda: R.stream_update(h, subs, 0.5, torch.bfloat16, 1e-5), nbytes=T * W * 18)
        add(f"poralorn: gated residual, split {T}x{W}",
            lambda: R.stream_update(h, subs, 0.5, torch.bfloat16, 1e-5, split=True), nbytes=T * W * 20)
        mixed, base = torch.randn(1, 2 * T, W, device=dev), torch.randn(1, T, W, device=dev)
        add(f"poralorn: entry of a pass + norm {T}x{W}", lambda: R.enter_pass(h, mixed, base, step, 1e-5),
            nbytes=T * W * 18)
        gu = rnd(T, 2 * I)
        add(f"uniform: swiglu {T}x{I}", lambda: dense.swiglu(gu), nbytes=T * I * 6)
        add(f"poralorn: exact GELU {T}x{I}", lambda: R.scaled_act(gu[:, :I], "gelu", one), nbytes=T * I * 4)


def _kernels_gumazen(b: _Bench) -> None:
    """The three kinds of attention with 32 heads of width 128 (4 key-value heads), the routed feed-forward with 120 + 8
    router outputs, and the row operations of two streams."""
    from ..models.decoder import _Init
    from ..models.hybrid import HybridBranch, RoutedFeedForward
    from ..models.moe import moe_forward
    from ..ops import dense, kv_cache
    from ..ops import moe as M
    from ..ops import rows as R
    from ..ops.attention import SeqInfo, attention_packed
    from ..ops.window_attention import QueryTiles, window_attention
    dev, add, rnd = torch.device("cuda"), b.add, _rnd
    W, H, G, D = 2048, 32, 4, 128
    base = get_config("gumazen-a3b")
    kinds = {"sink": base.hybrid.layers[1].branches[0], "window 1024": base.hybrid.layers[2].branches[0],
             "biases": base.hybrid.layers[0].branches[0]}
    gen = _Init(0, "cuda")
    branches = {k: HybridBranch(m, base, 0, 0, torch.bfloat16, "cuda", gen) for k, m in kinds.items()}

    def prepared(br):
        return copy.copy(br.prepare), {k: getattr(br, k).detach() for k in ("bias", "q_norm", "k_norm", "rel") if hasattr(br, k)}

    for n, L in ((8, 1024), (1, 8192)):
        T, nb = n * L, L // 64
        x = rnd(T, (H + 2 * G) * D)
        info = SeqInfo([L] * n, device=dev)
        flops = n * 4 * D * H * L * (L + 1) / 2
        add(f"uniform: fmha_fwd {n}x{L}", lambda: attention_packed(x, info, H, G, D), flops)
        table = torch.randperm(n * nb, device=dev).to(torch.int32).view(n, nb)
        cache = torch.zeros(n * nb, G * 64 * 2 * D, dtype=torch.bfloat16, device=dev)
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=dev)
        ids = torch.repeat_interleave(torch.arange(n, dtype=torch.int32), L).to(dev)
        pos = torch.arange(L, dtype=torch.int32).repeat(n).to(dev)
        tiles = QueryTiles([L] * n, [0] * n, list(range(n)), dev)
        tabs = dense.rope_tables(D, L, 1e6, device=dev)
        add(f"uniform: rotation + append {n}x{L}",
            lambda: kv_cache.rope_kv_append(x, pos, *tabs, None, ids, pos, table, cache.view(n * nb, 2, G, 64, D), H, G, D),
            nbytes=T * ((H + G) * D * 2 + (H + 2 * G) * D * 2))
        for name, br in branches.items():
            m, spec = br.b, br.spec
            xp = rnd(T, br.in_end)
            pr, w = prepared(br)
            for k, v in w.items():
                setattr(pr, k, v)
            add(f"gumazen: norms, rotation, append ({name}) {n}x{L}", lambda: pr.run(spec, xp, ids, pos, table, cache),
                nbytes=T * (H + 2 * G) * D * 4)
            seen = sum(min(i + 1, m.window) for i in range(L)) if m.window else L * (L + 1) / 2
            add(f"gumazen: attention ({name}) {n}x{L}, with norms, rotation, append",
                lambda: window_attention(spec, xp, ids, pos, table, cache, out, 0, tiles=tiles, prepare=pr),
                n * 4 * D * H * seen)
    for B, ctx in ((32, 2048), (256, 1024)):
        nb = (ctx + 63) // 64
        table = torch.randperm(B * nb, device=dev).to(torch.int32).view(B, nb)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        q, kvc = rnd(B, (H + 2 * G) * D), torch.zeros(B * nb, 2, G, 64, D, dtype=torch.bfloat16, device=dev)
        add(f"uniform: decode attention {B}x{ctx}", lambda: kv_cache.decode_attention(q, kvc, lens, table, H, G, D),
            nbytes=B * ctx * 2 * G * D * 2)
        flat, out = kvc.view(B * nb, -1), torch.empty(B, H * D, dtype=torch.bfloat16, device=dev)
        ids, pos = torch.arange(B, dtype=torch.int32, device=dev), lens - 1
        for name, br in branches.items():
            m, spec = br.b, br.spec
            xp = rnd(B, br.in_end)
            pr, w = prepared(br)
            for k, v in w.items():
                setattr(pr, k, v)
            add(f"gumazen: norms, rotation, append ({name}) {B}", lambda: pr.run(spec, xp, ids, pos, table, flat),
                nbytes=B * (H + 2 * G) * D * 4)
            seen = min(ctx, m.window) if m.window else ctx
            add(f"gumazen: decode attention ({name}) {B}x{ctx}, with norms, rotation, append",
                lambda: window_attention(spec, xp, ids, pos, table, flat, out, 0, seq_lens=lens, prepare=pr),
                nbytes=B * seen * 2 * G * D * 2)
    e = base.hybrid.layers[1].moe
    ff = RoutedFeedForward(e, W, 0.02, torch.bfloat16, "cuda", gen)
    router, local = rnd(e.experts, W), M.ExpertParallel()
    gu, dn = ff.gate_up_weight.detach(), ff.down_weight.detach()
    for T in (32, 256, 8192):
        x = rnd(T, W)
        used = e.experts * (1 - (1 - e.top / e.experts) ** T)
        flops, nbytes = T * e.top * 6.0 * W * e.ff, used * 6 * W * e.ff + T * W * 4
        z = torch.randn(1, T, e.outputs, device=dev)
        add(f"uniform: router {T}", lambda: M.route_topk(z[0, :, :e.experts].contiguous(), e.top), nbytes=T * e.outputs * 4)
        add(f"gumazen: router {T}", lambda: M.route_grouped(z, ff.correction.detach(), e.experts, e.top, e.groups, e.keep, e.scale),
            nbytes=T * e.outputs * 4)
        wt, ids = M.route_topk(z[0, :, :e.experts].contiguous(), e.top)
        add(f"uniform: routed feed-forward {T} (dispatch, experts, combine)",
            lambda: moe_forward(x, router, gu, dn, e.top, routed=(wt, ids)), flops, nbytes)
        i32 = ids.to(torch.int32)
        add(f"gumazen: routed feed-forward {T} (dispatch, experts)", lambda: M.routed_experts(x, i32, gu, dn, "silu"), flops, nbytes)
        h, y = torch.randn(T, 2, W, device=dev), rnd(1, T, W)
        conn = [torch.ones(2, device=dev).bfloat16(), torch.eye(2, device=dev).bfloat16(), rnd(W), rnd(W)]
        d, res, nw = rnd(T, W), rnd(T, W), rnd(W)
        add(f"uniform: residual + RMS norm {T}x{W} (bf16 stream)", lambda: dense.rmsnorm(d, nw, 1e-6, residual=res),
            nbytes=T * W * 8)
        kw = dict(w_in=conn[0], w_out=conn[0], w_mix=conn[1])
        add(f"gumazen: streams + layer norm {T}x{W} (two fp32 streams)",
            lambda: R.hyper_rows(h, conn[2], conn[3], 1e-5, result=R.SublayerSum(y), **kw), nbytes=T * W * 20)
        ys, slots = M.routed_experts(x, i32, gu, dn, "silu")
        w_id = torch.rand(T, device=dev)
        add(f"uniform: combine {T}x{W}", lambda: local.combine(ys, None, slots, wt, T, e.top), nbytes=T * W * 2 * (e.top + 1))
        add(f"gumazen: streams + layer norm + combine {T}x{W}",
            lambda: R.hyper_rows(h, conn[2], conn[3], 1e-5, result=R.SublayerSum(y, None, ys, slots, wt, x, w_id), **kw),
            nbytes=T * W * (22 + 2 * e.top))
        I = 11264
        up = rnd(T, 2 * I)
        add(f"uniform: swiglu {T}x{I}", lambda: dense.swiglu(up), nbytes=T * I * 6)
        add(f"gumazen: squared relu {T}x{I}", lambda: R.scaled_act(up[:, :I], "relu2"), nbytes=T * I * 4)


def _kernels_rizitar(b: _Bench) -> None:
    """Windowed attention with pooled runs (32 heads of width 128, 4 key-value heads), the delta rule with 32 heads of width 64
    beside the channel recurrence of the same size, the routed feed-forward with 120 plain experts, and the row operations."""
    from ..models.decoder import _Init
    from ..models.hybrid import HybridBranch
    from ..models.moe import moe_forward
    from ..ops import dense, kv_cache
    from ..ops import moe as M
    from ..ops import rows as R
    from ..ops.attention import SeqInfo, attention_packed
    from ..ops.recurrence import PortionPlan, RecurrenceSpec, empty_state, recurrence_decode, recurrence_prefill
    from ..ops.window_attention import QueryTiles, WindowSpec, window_attention
    dev, add, rnd = torch.device("cuda"), b.add, _rnd
    base = get_config("rizitar-a3b")
    W, H, G, D = base.hidden_size, 32, 4, 128
    gen = _Init(0, "cuda")
    kinds = [x.branches[0] for x in base.hybrid.layers]
    att = HybridBranch(next(m for m in kinds if m.kind == "attention"), base, 0, 0, torch.bfloat16, "cuda", gen)
    rule = HybridBranch(next(m for m in kinds if m.kind == "general_delta"), base, 0, 0, torch.bfloat16, "cuda", gen)
    m, spec = att.b, att.spec
    pr = copy.copy(att.prepare)
    for k in ("q_norm", "k_norm", "sink"):
        setattr(pr, k, getattr(att, k).detach())

    def seen(i):
        return min(i + 1, m.window) + max(0, i + 1 - m.window) // m.pool

    for n, L in ((8, 1024), (1, 8192)):
        T, nb, npool = n * L, L // 64, kv_cache.pool_blocks(L, m.pool)
        x, xp = rnd(T, (H + 2 * G) * D), rnd(T, att.in_end)
        info = SeqInfo([L] * n, device=dev)
        flops = n * 4 * D * H * L * (L + 1) / 2
        add(f"uniform: fmha_fwd {n}x{L}", lambda: attention_packed(x, info, H, G, D), flops)
        order = torch.randperm(n * (nb + npool), device=dev).to(torch.int32)
        table, pool_table = order[:n * nb].view(n, nb), order[n * nb:].view(n, npool).contiguous()
        cache = torch.zeros(n * (nb + npool), G * 64 * 2 * D, dtype=torch.bfloat16, device=dev)
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=dev)
        ids = torch.repeat_interleave(torch.arange(n, dtype=torch.int32), L).to(dev)
        pos = torch.arange(L, dtype=torch.int32).repeat(n).to(dev)
        tiles = QueryTiles([L] * n, [0] * n, list(range(n)), dev)
        tabs = dense.rope_tables(D, L, 1e6, device=dev)
        add(f"uniform: rotation + append {n}x{L}",
            lambda: kv_cache.rope_kv_append(x, pos, *tabs, None, ids, pos, table, cache[:n * nb].view(n * nb, 2, G, 64, D), H, G, D),
            nbytes=T * ((H + G) * D * 2 + (H + 2 * G) * D * 2))
        add(f"rizitar: norms, rotation, append, pooling {n}x{L}", lambda: pr.run(spec, xp, ids, pos, table, cache, pool_table),
            nbytes=T * (H + G) * D * 2 + T * (H + 2 * G) * D * 2 * (1 + 1 / m.pool))
        add(f"rizitar: attention window {m.window} pool {m.pool} {n}x{L}, with norms, rotation, append, pooling",
            lambda: window_attention(spec, xp, ids, pos, table, cache, out, 0, tiles=tiles, prepare=pr, pool_table=pool_table),
            n * 4 * D * H * sum(map(seen, range(L))))
        plain = WindowSpec(H, G, D, D, 0, H * D, (H + G) * D, D ** -0.5, m.window)
        add(f"domavik: window attention window {m.window} {n}x{L}, with append",
            lambda: window_attention(plain, x, ids, pos, table, cache, out, 0, tiles=tiles),
            n * 4 * D * H * sum(min(i + 1, m.window) for i in range(L)))
    for B, ctx in ((32, 2048), (256, 1024), (32, 16384)):
        nb, npool = (ctx + 63) // 64, kv_cache.pool_blocks(ctx, m.pool)
        order = torch.randperm(B * (nb + npool), device=dev).to(torch.int32)
        table, pool_table = order[:B * nb].view(B, nb), order[B * nb:].view(B, npool).contiguous()
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        flat = torch.zeros(B * (nb + npool), G * 64 * 2 * D, dtype=torch.bfloat16, device=dev)
        q, kvc = rnd(B, (H + 2 * G) * D), flat[:B * nb].view(B * nb, 2, G, 64, D)
        place = torch.randperm(B * nb, device=dev).to(torch.int32).view(B, nb)
        add(f"uniform: decode attention {B}x{ctx}", lambda: kv_cache.decode_attention(q, kvc, lens, place, H, G, D),
            nbytes=B * ctx * 2 * G * D * 2)
        out = torch.empty(B, H * D, dtype=torch.bfloat16, device=dev)
        ids, pos = torch.arange(B, dtype=torch.int32, device=dev), lens - 1
        xp = rnd(B, att.in_end)
        add(f"rizitar: norms, rotation, append, pooling {B} at {ctx}",
            lambda: pr.run(spec, xp, ids, pos, table, flat, pool_table, single=True),
            nbytes=B * (H + 2 * G) * D * 4 + B * m.pool * 2 * G * D * 2)
        add(f"rizitar: decode attention {B}x{ctx} window {m.window} pool {m.pool}, with norms, rotation, append, pooling",
            lambda: window_attention(spec, xp, ids, pos, table, flat, out, 0, seq_lens=lens, prepare=pr, pool_table=pool_table),
            nbytes=B * seen(ctx - 1) * 2 * G * D * 2)
        plain = WindowSpec(H, G, D, D, 0, H * D, (H + G) * D, D ** -0.5, m.window)
        add(f"domavik: window decode {B}x{ctx} window {m.window}, with append",
            lambda: window_attention(plain, q, ids, pos, table, flat, out, 0, seq_lens=lens),
            nbytes=B * min(ctx, m.window) * 2 * G * D * 2)
    d, h, spec = rule.b.dim, rule.b.heads, rule.spec
    hd = h * d
    chan = RecurrenceSpec("channel", h, d, d, 0, hd, 2 * hd, 3 * hd, 4 * hd, 0, 16, 16.0, 15.0, 1e-5, 1.0)
    for name, sp, wts, width in (
            ("rizitar: delta rule", spec, rule.weights(), rule.in_end),
            ("domavik: channel recurrence", chan, {"norm": rnd(d), "w2": rnd(hd, 16), "b_e": rnd(hd)}, 4 * hd + 16)):
        for n, L in ((8, 1024), (1, 8192)):
            x, out = rnd(n * L, width), torch.empty(n * L, hd, dtype=torch.bfloat16, device=dev)
            st, plan = empty_state(sp, n, dev), PortionPlan([L] * n, [0] * n, list(range(n)), dev)
            add(f"{name} {n}x{L} ({h} heads of {d})", lambda: recurrence_prefill(sp, x, wts, st, plan, out, 0),
                nbytes=n * L * (width + hd) * 2 + n * h * d * d * 4)
        for B in (32, 256):
            x, out = rnd(B, width), torch.empty(B, hd, dtype=torch.bfloat16, device=dev)
            st = empty_state(sp, B, dev)
            slots, pos = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), 9, dtype=torch.int32, device=dev)
            add(f"{name} step {B} ({h} heads of {d})", lambda: recurrence_decode(sp, x, wts, st, slots, pos, out, 0),
                nbytes=B * h * d * d * 8 + B * (width + hd) * 2)
    e = next(x.moe for x in base.hybrid.layers if x.moe is not None)
    wide, local, one = e.ff * 2 // 3, M.ExpertParallel(), rnd(W)
    up, dn = rnd(e.experts, e.ff, W) * 0.04, rnd(e.experts, W, e.ff) * 0.04
    gu, gd, router = rnd(e.experts, 2 * wide, W) * 0.04, rnd(e.experts, W, wide) * 0.04, rnd(e.experts, W)
    side, numbers = base.hybrid.token_side, torch.tensor([0.5, 0.3], device=dev).bfloat16()
    table = rnd(base.vocab_size, 4 * side)
    for T in (32, 256, 8192):
        x, z = rnd(T, W), torch.randn(1, T, e.experts, device=dev)
        used = e.experts * (1 - (1 - e.top / e.experts) ** T)
        flops, nbytes = T * e.top * 4.0 * W * e.ff, used * 4 * W * e.ff + T * W * 4
        add(f"uniform: router {T}", lambda: M.route_topk(z[0], e.top, False), nbytes=T * e.experts * 4)
        add(f"rizitar: router {T}", lambda: M.route_grouped(z, None, e.experts, e.top, 1, 1, 1.0, outputs=e.experts,
                                                            renormalize=False), nbytes=T * e.experts * 4)
        wt, ids = M.route_topk(z[0], e.top, False)
        add(f"uniform: routed feed-forward {T} (dispatch, gated experts, combine)",
            lambda: moe_forward(x, router, gu, gd, e.top, routed=(wt, ids)), flops, nbytes)
        i32 = ids.to(torch.int32)
        add(f"rizitar: routed feed-forward {T} (dispatch, plain experts)",
            lambda: M.routed_experts(x, i32, up, dn, "relu2", gated=False), flops, nbytes)
        h32, y, d16, res = torch.randn(T, W, device=dev), rnd(1, T, W), rnd(T, W), rnd(T, W)
        add(f"uniform: residual + RMS norm {T}x{W} (bf16 stream)", lambda: dense.rmsnorm(d16, one, 1e-6, residual=res),
            nbytes=T * W * 8)
        add(f"rizitar: norm, residual, norm {T}x{W} (fp32 stream)",
            lambda: R.post_norm_rows(h32, one, 1e-5, torch.bfloat16, post=one, result=R.SublayerSum(y)), nbytes=T * W * 12)
        ys, slots = M.routed_experts(x, i32, up, dn, "relu2", gated=False)
        add(f"uniform: combine {T}x{W}", lambda: local.combine(ys, None, slots, wt, T, e.top), nbytes=T * W * 2 * (e.top + 1))
        add(f"rizitar: combine, norm, residual, norm {T}x{W}",
            lambda: R.post_norm_rows(h32, one, 1e-5, torch.bfloat16, post=one,
                                     result=R.SublayerSum(ys=ys, pair_slot=slots, pair_w=wt)), nbytes=T * W * (10 + 2 * e.top))
        tok, zs = torch.randint(0, base.vocab_size, (T,), device=dev), rnd(1, T, side)
        add(f"uniform: swiglu {T}x{side}", lambda: dense.swiglu(torch.cat([zs[0], zs[0]], 1)), nbytes=T * side * 6)
        add(f"rizitar: token gate {T}x{side}", lambda: R.token_gate(zs, tok, table, side, side, torch.bfloat16),
            nbytes=T * side * 6)
        I = base.intermediate_size
        a, bias = rnd(1, T, I), rnd(I)
        pair = rnd(T, 2 * I)
        add(f"uniform: swiglu {T}x{I}", lambda: dense.swiglu(pair), nbytes=T * I * 6)
        add(f"rizitar: bias + xIELU {T}x{I}", lambda: R.bias_act(a, "xielu", torch.bfloat16, bias=bias, numbers=numbers),
            nbytes=T * I * 4)


def _kernels_domavik(b: _Bench) -> None:
    from ..ops import dense, kv_cache
    from ..ops import rows as R
    from ..ops.attention import SeqInfo, attention_packed
    from ..ops.recurrence import PortionPlan, RecurrenceSpec, empty_state, recurrence_decode, recurrence_prefill
    from ..ops.window_attention import QueryTiles, WindowSpec, window_attention
    dev, add, rnd = torch.device("cuda"), b.add, _rnd
    # attention on prompts: 28 heads, 4 kv heads, width 128
    H, G, D = 28, 4, 128
    for n, L in ((8, 1024), (1, 8192)):
        T = n * L
        x = rnd(T, (H + 2 * G) * D)
        info = SeqInfo([L] * n, device=dev)
        flops = n * 4 * D * H * L * (L + 1) / 2
        add(f"uniform: fmha_fwd {n}x{L}", lambda: attention_packed(x, info, H, G, D), flops)
        nb = L // 64
        table = torch.randperm(n * nb, device=dev).to(torch.int32).view(n, nb)
        cache = torch.zeros(n * nb, G * 64 * 2 * D, dtype=torch.bfloat16, device=dev)
        out = torch.empty(T, H * D, dtype=torch.bfloat16, device=dev)
        ids = torch.repeat_interleave(torch.arange(n, dtype=torch.int32), L).to(dev)
        pos = torch.arange(L, dtype=torch.int32).repeat(n).to(dev)
        tiles = QueryTiles([L] * n, [0] * n, list(range(n)), dev)
        for w, kf in ((0, 0), (1024, 64)):
            spec = WindowSpec(H, G, D, D, 0, H * D, (H + G) * D, D ** -0.5, w, kf, 8.0)
            seen = sum(min(i + 1, w) + max(0, min(kf, i + 1 - w)) for i in range(L)) if w else L * (L + 1) / 2
            add(f"domavik: window attention {n}x{L} window {w or 'none'} (with cache append)",
                lambda: window_attention(spec, x, ids, pos, table, cache, out, 0, tiles=tiles), n * 4 * D * H * seen)
    # attention on single tokens
    for B, ctx in ((32, 2048), (256, 1024)):
        nb = (ctx + 63) // 64
        table = torch.randperm(B * nb, device=dev).to(torch.int32).view(B, nb)
        cache = torch.zeros(B * nb, 2, G, 64, D, dtype=torch.bfloat16, device=dev)
        x = rnd(B, (H + 2 * G) * D)
        lens = torch.full((B,), ctx, dtype=torch.int32, device=dev)
        add(f"uniform: decode attention {B}x{ctx}", lambda: kv_cache.decode_attention(x, cache, lens, table, H, G, D),
            nbytes=B * ctx * 2 * G * D * 2)
        out = torch.empty(B, H * D, dtype=torch.bfloat16, device=dev)
        ids, pos = torch.arange(B, dtype=torch.int32, device=dev), lens - 1
        flat = cache.view(B * nb, -1)
        for w, kf in ((0, 0), (1024, 64)):
            spec = WindowSpec(H, G, D, D, 0, H * D, (H + G) * D, D ** -0.5, w, kf, 8.0)
            seen = min(ctx, w) + max(0, min(kf, ctx - w)) if w else ctx
            add(f"domavik: window decode {B}x{ctx} window {w or 'none'} (with cache append)",
                lambda: window_attention(spec, x, ids, pos, table, flat, out, 0, seq_lens=lens),
                nbytes=B * seen * 2 * G * D * 2)
    # recurrences
    for gate, h, dk, dv in (("channel", 16, 64, 128), ("head", 16, 128, 128)):
        up, at, off = (lambda n: (n + 7) // 8 * 8), 0, {}
        for key, wd in (("q", h * dk), ("k", h * dk), ("v", h * dv), ("g", h * dv)) + (
                (("e", 16),) if gate == "channel" else (("e", h), ("f", h))):
            off[key], at = at, at + up(wd)
        spec = RecurrenceSpec(gate, h, dk, dv, off["q"], off["k"], off["v"], off["g"], off["e"], off.get("f", 0),
                              16 if gate == "channel" else 0, 16.0, 15.0, 1e-5, 1.0,
                              "silu" if gate == "channel" else "sigmoid", gate == "head")
        wts = {"norm": rnd(h * dv if gate == "head" else dv)}
        wts.update({"w2": rnd(h * dk, 16), "b_e": rnd(h * dk)} if gate == "channel" else {"b_e": rnd(h), "b_f": rnd(h) + 3})
        for n, L in ((8, 1024), (1, 8192)):
            x = rnd(n * L, at)
            out = torch.empty(n * L, h * dv, dtype=torch.bfloat16, device=dev)
            st = empty_state(spec, n, dev)
            plan = PortionPlan([L] * n, [0] * n, list(range(n)), dev)
            nbytes = n * L * (at + h * dv) * 2 + n * h * spec.rows * dk * 4
            flops = n * L * h * 2.0 * dk * dv * 2
            add(f"domavik: {gate} recurrence {n}x{L}", lambda: recurrence_prefill(spec, x, wts, st, plan, out, 0), flops,
                nbytes)
        for B in (32, 256):
            x = rnd(B, at)
            out = torch.empty(B, h * dv, dtype=torch.bfloat16, device=dev)
            st = empty_state(spec, B, dev)
            slots, pos = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), 9, dtype=torch.int32, device=dev)
            add(f"domavik: {gate} recurrence step {B}",
                lambda: recurrence_decode(spec, x, wts, st, slots, pos, out, 0), nbytes=B * h * spec.rows * dk * 8)
    # row operations
    for T in (256, 8192):
        W, I, V = 3584, 18944, 152064
        h32, d, w = torch.randn(T, W, device=dev), rnd(T, W), rnd(W)
        res = rnd(T, W)
        add(f"uniform: residual + RMS norm {T}x{W} (bf16 stream)", lambda: dense.rmsnorm(d, w, 1e-6, residual=res),
            nbytes=T * W * 8)
        add(f"domavik: residual + layer norm {T}x{W} (fp32 stream)", lambda: R.add_norm(h32, d, w, 1e-5),
            nbytes=T * W * 12)
        gu = rnd(T, 2 * I)
        add(f"uniform: swiglu {T}x{I}", lambda: dense.swiglu(gu), nbytes=T * I * 6)
        add(f"domavik: gelu gate {T}x{I}", lambda: R.gated_act(gu), nbytes=T * I * 6)
        ids = torch.randint(0, V, (T,), device=dev)
        table = torch.zeros(V, W, dtype=torch.bfloat16, device=dev)
        add(f"uniform: embedding {T}x{W}", lambda: dense.embedding(ids, table), nbytes=T * W * 4)
        add(f"domavik: scaled embedding {T}x{W}", lambda: R.embed_scaled(ids, table, 2.0), nbytes=T * W * 6)
        if T == 256:
            z = torch.randn(T, V, device=dev)
            add(f"domavik: soft cap {T}x{V}", lambda: R.softcap_(z, 30.0), nbytes=T * V * 8)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--only", default="", help="kernels whose name contains this")
    ap.add_argument("--iters", type=int, default=20)
    ap.add_argument("--design", choices=list(SIZES), default="domavik")
    ap.add_argument("--sizes", default="", help="comma separated, default all of the design")
    args = ap.parse_args(argv)
    res = kernels(args.design, args.only, args.iters) if args.kernels else serve(
        args.design, args.sizes.split(",") if args.sizes else None)
    print(json.dumps(res), flush=True)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
