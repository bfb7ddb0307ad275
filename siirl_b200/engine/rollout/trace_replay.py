"""Teacher-forced replay of request batches through the rollout engine.

The engine's own prefill and decode forward, block allocator, slots and recurrent states run on given token ids instead
of sampled ones, step by step, and the logits at chosen places are written out: for comparing checkpoints or builds, or
for scoring a recorded conversation the way it was served.

One step is one JSON line

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: the next tokens of each request and the places among them whose logits are wanted; ``end``: requests that
are finished after the step.  The first tokens of a request, and any later portion of more than one token, run as
prompt portions (one packed batch); requests that go on by one token run as one decode step.  ``OUT/<step>.f32`` gets
the wanted logits (little-endian fp32, entries' order) and ``done <step>`` is printed after every step."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Sequence, Tuple

import torch

from .native_engine import BLOCK, RolloutEngine, _Seq


class TraceReplay:
    def __init__(self, engine: RolloutEngine, max_slots: int = 16):
        self.engine = engine
        self.max_slots = max_slots
        self.live: Dict[str, _Seq] = {}
        self.free: List[int] = []

    def _place(self, n_new: int) -> None:
        """Room for ``n_new`` more requests; the slot count only changes while nothing is live."""
        eng = self.engine
        if not self.live and (eng.num_slots < n_new or eng.num_slots == 0):
            eng._ensure_slots(max(self.max_slots, (n_new + 7) // 8 * 8))
            eng._reset_slots()
            self.free = list(range(eng.num_slots))[::-1]
        if len(self.free) < n_new:
            raise RuntimeError(f"{len(self.live)} live requests and {n_new} new ones exceed {eng.num_slots} slots")

    def _grow(self, seq: _Seq, tokens: int) -> bool:
        """Blocks for positions below ``tokens``; true when the block table changed."""
        need = (tokens + BLOCK - 1) // BLOCK
        if need > self.engine.max_blocks_per_seq:
            raise ValueError(f"{tokens} tokens exceed the engine's max_model_len {self.engine.max_model_len}")
        before = len(seq.blocks), len(seq.pool_blocks)
        while len(seq.blocks) < need:
            seq.blocks.append(self.engine.alloc.alloc())
        while len(seq.pool_blocks) < self.engine._pool_blocks_needed(tokens):
            seq.pool_blocks.append(self.engine.alloc.alloc())
        return (len(seq.blocks), len(seq.pool_blocks)) != before

    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[str, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """``(id, tokens, want)`` per request; returns the wanted fp32 logits ``[sum of wants, vocab]`` on the CPU."""
        eng, dev = self.engine, self.engine.device
        vocab = eng.cfg.vocab_size
        new = [e for e in entries if e[0] not in self.live]
        self._place(len(new))
        for rid, _, _ in new:
            self.live[rid] = _Seq(0, 0, 0, 0, slot=self.free.pop())
        jobs, grown = [], []
        for rid, tokens, want in entries:
            seq = self.live[rid]
            if any(not 0 <= t < vocab for t in tokens) or any(not 0 <= w < len(tokens) for w in want):
                raise ValueError(f"request {rid}: token id or wanted place out of range")
            if self._grow(seq, seq.prefilled + len(tokens)):
                grown.append(seq)
            jobs.append((seq, list(tokens), list(want)))
        if grown:
            eng._write_block_tables(grown)
        out: List[torch.Tensor] = [torch.empty(0, vocab)] * len(jobs)

        portions = [k for k, (s, t, _) in enumerate(jobs) if t and (len(t) > 1 or s.prefilled == 0)]
        if portions:
            hidden = eng._prefill([jobs[k][0] for k in portions], [jobs[k][1] for k in portions],
                                  [jobs[k][0].prefilled for k in portions], all_rows=True)
            rows, at = [], 0
            for k in portions:
                rows += [at + w for w in jobs[k][2]]
                at += len(jobs[k][1])
            if rows:
                z = eng._logits(hidden.index_select(0, torch.tensor(rows, device=dev))).cpu()
                for k, part in zip(portions, z.split([len(jobs[k][2]) for k in portions])):
                    out[k] = part
        singles = [k for k, (s, t, _) in enumerate(jobs) if len(t) == 1 and k not in portions]
        if singles:
            slots = torch.tensor([jobs[k][0].slot for k in singles], dtype=torch.int64, device=dev)
            eng.ctx_len[slots] = torch.tensor([jobs[k][0].prefilled for k in singles], dtype=torch.int32, device=dev)
            eng.last_token[slots] = torch.tensor([jobs[k][1][0] for k in singles], dtype=torch.int64, device=dev)
            eng.finished.fill_(True)
            eng.finished[slots] = False
            z = eng._decode_logits()
            eng.finished.fill_(True)
            wanted = [k for k in singles if jobs[k][2]]
            if wanted:
                z = z.index_select(0, torch.tensor([jobs[k][0].slot for k in wanted], device=dev)).cpu()
                for i, k in enumerate(wanted):
                    out[k] = z[i:i + 1].expand(len(jobs[k][2]), -1)
        for seq, tokens, _ in jobs:
            seq.prefilled += len(tokens)
            eng._release_hidden_blocks(seq, seq.prefilled)
        if dev.type == "cuda":
            from ...ops import lib
            lib.check_status(dev)
        return torch.cat(out) if out else torch.empty(0, vocab)

    def end(self, rids: Sequence[str]) -> None:
        for rid in rids:
            seq = self.live.pop(rid)
            self.engine._release_blocks(seq)
            self.engine._clear_tables(seq.slot)
            self.free.append(seq.slot)


def load_engine(path: str, dtype: torch.dtype, max_tokens: int, slots: int = 16, device="cuda") -> RolloutEngine:
    from ...models.config import get_config
    from ...models.decoder import build_model
    from ...models.hf_io import load_hf_weights
    cfg = get_config(path)
    model = build_model(cfg, dtype=dtype, device=device)
    load_hf_weights(model, path)
    for p in model.parameters():
        p.requires_grad_(False)
    # every live request may end in a partly filled block
    blocks = (max_tokens + BLOCK - 1) // BLOCK + 64 + slots
    pools = cfg.hybrid.pools() if cfg.hybrid is not None else []
    if pools:       # one more entry per run of tokens, in blocks that may be partly filled too
        blocks += max_tokens // (pools[0] * BLOCK) + 1 + slots
    return RolloutEngine(model, max_num_seqs=slots, max_model_len=max_tokens + BLOCK, num_blocks=blocks)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay request batches through the serving engine")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16",
                    help="bfloat16: the serving kernels; float32: true 32-bit everywhere (hybrid decoders)")
    ap.add_argument("--out", required=True, help="folder that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=65536, help="most tokens live requests hold at any time")
    args = ap.parse_args(argv)
    dtype = getattr(torch, args.dtype)
    from ...models.config import get_config
    if dtype == torch.float32 and get_config(args.model).hybrid is None:
        print("trace_run: this model family runs in bfloat16 only", file=sys.stderr)
        return 3
    from ...ops import lib
    lib.use_serving_library()       # compiled on first use in a fresh checkout
    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a GPU")
    torch.backends.cuda.matmul.allow_tf32 = False
    replay = TraceReplay(load_engine(args.model, dtype, args.max_tokens))
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        z = replay.step([(e["id"], e["tokens"], e.get("want", [])) for e in msg["entries"]])
        if z.shape[0]:
            with open(os.path.join(args.out, f"{msg['step']}.f32"), "wb") as f:
                f.write(z.contiguous().numpy().astype("<f4").tobytes())
        replay.end(msg.get("end", []))
        print(f"done {msg['step']}", flush=True)
    return 0
