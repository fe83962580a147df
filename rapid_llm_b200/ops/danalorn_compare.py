"""Prefill and decode throughput of Danalorn models at layer sizes of real models, beside Basitar and Qwen3 of equal width
and depth, and the kernels that came with the design (or got a new form for it) alone, each next to the like kernel of the
closest model in the same harness.

    python bench.py --workload danalorn [--sizes 2048,4096]
    python -m rapid_llm_b200.ops.danalorn_compare [--sizes 2048,4096]
    python -m rapid_llm_b200.ops.danalorn_compare --alone --sizes 2048      # the kernels a few times each, for ncu

Random weights, bfloat16, one GPU.  A model of width ``W`` has six layers, ``latent_attention, gla, latent_attention`` (which
reads the first one's rows)``, attention, gla, gla``, each with a squared-relu feed-forward of ``4 W``: ``W / 128`` latent
heads of 128 plain, 64 rotated and 128 value entries over a latent of 192 (a cached row of 256 numbers) and a query latent of
``3 W / 8`` with a window of 512; ``W / 128`` query heads of 128 over ``W / 512`` key/value heads; ``W / 64`` recurrent heads
of 64 with a decay product of rank 16.  Basitar beside it has the same latent and recurrent sizes in the order
``latent_attention, wkv, latent_attention, latent_attention_2, wkv, wkv`` with a gated feed-forward of ``8 W / 3`` (the same
number of weights) in every layer; Qwen3 has six layers of the same width.  Prefill is one 2,048-token step (best of three,
CUDA events around the step function); decode is batch 8 behind 1,024-token prompts, replayed from the captured graph (median
of 32 steps).  Kernels are timed alone with CUDA events, L2 flushed between runs (a write of 256 MB), on one 2,048-token
prompt and on 64 single tokens behind 1,024 cached ones; ``frac`` is (bytes the kernel must move) / time / measured copy
bandwidth, ``tflops`` the products' arithmetic over the same time.
"""

from __future__ import annotations

import argparse
import json
import statistics
from types import SimpleNamespace

import torch

from .basitar_compare import KV_RANK, PLAIN, ROT, VDIM, WKV_DIM, basitar_raw
from .recurrent_compare import PREFILL, _events, model_figures, qwen3_raw

WINDOW, RANK, TAU = 512, 16, 16.0


def danalorn_raw(width: int) -> dict:
    heads = width // 128
    latent = {"heads": heads, "dim": PLAIN, "rot_dim": ROT, "vdim": VDIM, "kv_rank": KV_RANK, "q_rank": 3 * width // 8,
              "rot": {"base": 1.0e4, "dims": ROT}, "scale": (PLAIN + ROT) ** -0.5, "mask": {"size": WINDOW}}
    soft = {"heads": heads, "kv_heads": max(heads // 4, 1), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
            "q_temp": {"coef": 0.1, "every": 8192}}
    gla = {"heads": width // WKV_DIM, "dim": WKV_DIM, "vdim": WKV_DIM, "tau": TAU, "decay_rank": RANK}
    order = [("latent_attention", latent), ("gla", gla), ("latent_attention", {**latent, "kv_from": 0}), ("attention", soft), ("gla", gla), ("gla", gla)]
    return {"architecture": "Danalorn", "vocab": 32000, "width": width, "norm": {"eps": 1e-6},
            "embedding": {"scale": 1.0, "bigram": {"buckets": 65521, "mul_prev": 31, "mul_cur": 17}},
            "layers": [{"type": kind, "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": 4 * width}} for kind, mixer in order]}


def dense_basitar_raw(width: int) -> dict:
    raw = basitar_raw(width)
    by_type = {layer["type"]: layer for layer in raw["layers"]}
    dense = {"kind": "dense", "ff": (8 * width // 3 + 255) // 256 * 256}
    raw["layers"] = [{**by_type[kind], "mlp": dict(dense)} for kind in
                     ("latent_attention", "wkv", "latent_attention", "latent_attention_2", "wkv", "wkv")]
    return raw


def kernel_figures(width: int, hbm_gbs: float) -> dict:
    """The design's own kernels alone, and beside each the like kernel of the closest model, on a 2,048-token prompt and
    on single tokens."""
    import numpy as np

    from ..parts.attention import AttentionItems
    from ..parts.base import StepShape
    from . import gemm, kernels

    device = "cuda:0"
    heads, kv_heads, d, wide_d, q_rank = width // 128, max(width // 512, 1), 128, 256, 3 * width // 8
    flush = torch.empty(64 << 20, dtype=torch.float32, device=device)
    out = {}

    def timed(label, tokens, entries, moved, run, flops=0.0):
        times = []
        for _ in range(7):
            flush.zero_()
            begin, end = _events()
            begin.record()
            run()
            end.record()
            torch.cuda.synchronize()
            times.append(begin.elapsed_time(end) * 1e3)
        us = statistics.median(times[2:])
        row = {"us": round(us, 1), "mb": round(moved / 1e6, 2), "frac": round(moved / (us * 1e-6) / (hbm_gbs * 1e9), 3)}
        if flops:
            row["tflops"] = round(flops / (us * 1e-6) / 1e12, 1)
        out[f"{label} ({'prompt of ' + str(tokens) if entries == 1 else str(entries) + ' single tokens'})"] = row

    bf = lambda *shape: torch.randn(*shape, device=device).to(torch.bfloat16)      # noqa: E731
    f32 = lambda *shape: torch.randn(*shape, device=device)                        # noqa: E731
    fault = torch.zeros(1, dtype=torch.int32, device=device)
    page, context = 16, 1024
    for tokens, entries in ((PREFILL, 1), (64, 64)):
        per, start = tokens // entries, 0 if entries == 1 else context
        positions = (start + torch.arange(per, dtype=torch.int32, device=device)).repeat(entries)
        batch = SimpleNamespace(
            token_ids=torch.randint(0, 32000, (tokens,), dtype=torch.int32, device=device), feedback=None, positions=positions,
            cu_seqlens=torch.arange(0, tokens + 1, per, dtype=torch.int32, device=device),
            entry_slot=torch.arange(entries, dtype=torch.int32, device=device),
            entry_start=torch.full((entries,), start, dtype=torch.int32, device=device), num_entries=entries, fault=fault)
        pages_per = -(-(start + per) // page)
        table = (1 + torch.arange(entries * pages_per, dtype=torch.int32, device=device)).view(entries, pages_per)
        slot_of = torch.arange(entries, dtype=torch.int32, device=device).repeat_interleave(per)
        dest = (table[slot_of.long(), (positions // page).long()] * page + positions % page).to(torch.int32)
        step = StepShape(lengths=np.full(entries, per, dtype=np.int32), starts=np.full(entries, start, dtype=np.int32),
                         decode_only=per == 1, page_size=page)
        # -- the embedding: scaled token row and pair row, beside the sum with a position row
        embed, pair, place = bf(32000, width), bf(65522, width), bf(4096, width)
        rows, stream = torch.empty(tokens, width, dtype=torch.bfloat16, device=device), f32(tokens, width)
        last = torch.zeros(entries, 1, dtype=torch.int32, device=device)
        timed("embedding_sum, scaled, no positions", tokens, entries, tokens * width * 10,
              lambda: kernels.embedding_sum(rows, stream, embed, pair, None, batch, last, mul_prev=31, mul_cur=17, scale=2.0))
        timed("embedding_sum (like kernel)", tokens, entries, tokens * width * 12,
              lambda: kernels.embedding_sum(rows, stream, embed, pair, place, batch, last, mul_prev=31, mul_cur=17))
        # -- per-head norm with a temperature and no rotation on rows that hold the gate too, beside the rotating kernel
        qkv_width = (heads + 2 * kv_heads) * d
        wide, plain = bf(tokens, qkv_width + heads * d), bf(tokens, qkv_width)
        q = torch.empty(tokens, heads * d, dtype=torch.bfloat16, device=device)
        cache = torch.zeros(entries * pages_per + 1, 2, kv_heads, page, d, dtype=torch.bfloat16, device=device)
        cache.normal_()
        weight = 1 + 0.1 * f32(d)
        nothing, angles = torch.empty(4096, 0, device=device), f32(4096, d // 2)
        common = {"num_heads": heads, "num_kv_heads": kv_heads, "head_dim": d, "positions": positions, "eps": 1e-6, "fault": fault,
                  "q_weight": weight, "k_weight": weight, "kv_dest": dest, "cache": cache, "page_size": page}
        timed("qk_norm_write, temperature, no rotation", tokens, entries, tokens * qkv_width * 4,
              lambda: kernels.qk_norm_rope_write(wide, q, rotary_dim=0, cos=nothing, sin=nothing, temperature=(0.1, 512.0), **common))
        timed("qk_norm_rope_write (like kernel)", tokens, entries, tokens * qkv_width * 4,
              lambda: kernels.qk_norm_rope_write(plain, q, rotary_dim=d, cos=angles, sin=angles, **common))
        # -- attention with slopes and the fixed sink, beside the plain one
        q.normal_()
        attended = torch.empty_like(q)
        plan = AttentionItems(heads // kv_heads, kv_heads, d).plan(step)
        items = {name: torch.from_numpy(plan[name]).to(device) for name in ("chunk_items", "decode_items")}
        splits = plan["splits"]
        part_out = torch.empty(tokens * heads * splits, d, device=device) if splits > 1 else None
        part_lse = torch.empty(tokens * heads * splits, 1, device=device) if splits > 1 else None
        slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], device=device)
        one = torch.zeros(heads, device=device)
        keys = sum(range(start + 1, start + per + 1)) * entries
        moved = entries * (start + per) * kv_heads * d * 4 + tokens * heads * d * 4
        for label, extra in (("attention, slopes, fixed sink", {"slopes": slopes, "sink": one}), ("attention (like kernel)", {})):
            timed(label, tokens, entries, moved, lambda extra=extra: kernels.attention_mma(
                q, cache, attended, splits=splits, part_out=part_out, part_lse=part_lse, cu_seqlens=batch.cu_seqlens,
                entry_start=batch.entry_start, entry_slot=batch.entry_slot, block_table=table, num_heads=heads, num_kv_heads=kv_heads,
                head_dim=d, window=0, scale=d ** -0.5, fault=fault, decode_rows=plan["decode_rows"], chunk_rows=plan["chunk_rows"],
                decode_splits=plan["decode_splits"], **items, **extra), flops=4.0 * keys * heads * d)
        gated = torch.empty_like(q)
        timed("sigmoid_gate, entry by entry", tokens, entries, tokens * heads * d * 6,
              lambda: kernels.sigmoid_gate(attended, wide[:, qkv_width:], gated))
        # -- latents: a query latent alone, beside both latents and the cache row
        down = bf(tokens, q_rank + wide_d)
        rows_cache = torch.zeros(entries * pages_per + 1, page, wide_d, dtype=torch.bfloat16, device=device)
        rows_cache.normal_()
        c_q = torch.empty(tokens, q_rank, dtype=torch.bfloat16, device=device)
        q_weight, c_weight, freq = f32(q_rank), f32(KV_RANK), torch.rand(ROT // 2, device=device)
        shape = {"q_col0": 0, "q_rank": q_rank, "c_col0": q_rank, "kv_rank": KV_RANK, "rot": ROT, "q_weight": q_weight, "eps": 1e-6, "q_out": c_q,
                 "positions": positions, "freq": freq, "magnitude": 1.0, "layout": kernels.ROTATE_NEIGHBOURS, "fault": fault}
        timed("latent_norm_write, query latent alone", tokens, entries, tokens * q_rank * 4,
              lambda: kernels.latent_norm_write(down, c_weight=None, cache=None, kv_dest=None, **shape))
        timed("latent_norm_write (like kernel)", tokens, entries, tokens * (q_rank + wide_d) * 4,
              lambda: kernels.latent_norm_write(down, c_weight=c_weight, cache=rows_cache, kv_dest=dest, **shape))
        # -- attention over one cached row a token with a window and a sink, beside all keys
        wide_q = bf(tokens, heads * wide_d)
        wide_out = torch.empty_like(wide_q)
        sink = f32(heads)
        for label, window, term in (("attention over cached rows, window of 512, sink", WINDOW, sink), ("attention over cached rows, all keys (like kernel)", 0, None)):
            plan = AttentionItems(heads, 1, wide_d, tensor_core=False, window=window).plan(step)
            items = {name: torch.from_numpy(plan[name]).to(device) for name in ("chunk_items", "decode_items")}
            splits = plan["splits"]
            part_out = torch.empty(tokens * heads * splits, wide_d, device=device) if splits > 1 else None
            part_lse = torch.empty(tokens * heads * splits, 1, device=device) if splits > 1 else None
            reach = window or 1 << 30
            keys = sum(min(p, reach) for p in range(start + 1, start + per + 1)) * entries
            moved = entries * min(start + per, per + reach) * wide_d * 2 + tokens * heads * wide_d * 4
            timed(label, tokens, entries, moved, lambda: kernels.attention_mma(
                wide_q, rows_cache.view(-1, 1, 1, page, wide_d), wide_out, splits=splits, part_out=part_out, part_lse=part_lse,
                cu_seqlens=batch.cu_seqlens, entry_start=batch.entry_start, entry_slot=batch.entry_slot, block_table=table, num_heads=heads,
                num_kv_heads=1, head_dim=wide_d, window=window, scale=(PLAIN + ROT) ** -0.5, fault=fault, sink=term, decode_kernel="mma",
                decode_rows=plan["decode_rows"], chunk_rows=kernels.CHUNK_TILE_ROWS, **items), flops=4.0 * keys * heads * wide_d)
        # -- the recurrent mixer: decays from the low-rank rows with q, k and v as float32, beside wkv's three kernels
        c, rec_heads = width, width // WKV_DIM
        proj = bf(tokens, 4 * c + RANK)
        a2, a_bias = bf(c, RANK), f32(c)
        qkv, decay = f32(tokens, 3 * c), f32(tokens, c)
        timed("low_rank_decay, q, k and v as float32", tokens, entries, tokens * (3 * c * 6 + RANK * 2 + c * 4) + a2.numel() * 2,
              lambda: kernels.low_rank_decay(proj[:, : 3 * c], proj[:, 4 * c :], a2, a_bias, TAU, qkv, decay))
        high, w0 = proj[:, :c], f32(c)
        timed("exp_decay (like kernel)", tokens, entries, tokens * c * 6, lambda: kernels.exp_decay(high, w0, decay))
        timed("activate_rows, q, k and v as float32 (like kernel)", tokens, entries, tokens * 3 * c * 6,
              lambda: kernels.activate_rows(proj[:, : 3 * c], qkv, act=False))
        low = bf(tokens, 64)
        w2 = bf(c, 64)
        z = torch.empty(tokens, c, dtype=torch.bfloat16, device=device)
        timed("second product of a low-rank pair (like kernel)", tokens, entries, (low.numel() + w2.numel() + z.numel()) * 2,
              lambda: gemm.linear(low, w2, z, fault))
        decay.uniform_(0.9, 1.0)
        qkv.normal_()
        state = torch.zeros(entries, rec_heads * WKV_DIM * WKV_DIM, device=device)
        read, bonus = f32(tokens, c), f32(rec_heads, WKV_DIM)
        for label, extra in (("linear_scan, row decays", {}), ("linear_scan, row decays and a bonus (like kernel)", {"bonus": bonus})):
            timed(label, tokens, entries, 2 * state.numel() * 4 + 5 * tokens * c * 4, lambda extra=extra: kernels.linear_scan(
                qkv[:, :c], qkv[:, c : 2 * c], qkv[:, 2 * c :], decay, read, state, batch, heads=rec_heads, kv_heads=rec_heads, dim=WKV_DIM,
                vdim=WKV_DIM, **extra))
        normed, head_weight, column_weight = torch.empty(tokens, c, dtype=torch.bfloat16, device=device), f32(WKV_DIM), f32(c)
        for label, w in (("gated_norm, one weight for all heads", head_weight), ("gated_norm, a weight per column (like kernel)", column_weight)):
            timed(label, tokens, entries, tokens * c * 8, lambda w=w: kernels.gated_norm(
                read, normed, group=WKV_DIM, gate=proj[:, 3 * c : 4 * c], act=kernels.GATE_SILU, weight=w, eps=1e-6))
    assert int(fault.item()) == 0, "a kernel reported a fault"
    return out


def alone(width: int = 2048) -> None:
    """Every kernel of :func:`kernel_figures` a few times and nothing else: the case a profiler captures, picking its
    kernel by name."""
    kernel_figures(width, 6650.0)
    torch.cuda.synchronize()


def run(sizes: list[int], hbm_gbs: float) -> dict:
    from ..config import BasitarConfig, DanalornConfig, Qwen3Config

    result = {"workload": "danalorn beside basitar and qwen3, equal sizes", "dtype": "bf16", "data": "synthetic",
              "prefill_tokens": PREFILL, "decode_batch": 8, "decode_context": 1024, "sizes": {}}
    for width in sizes:
        result["sizes"][str(width)] = {
            "danalorn": model_figures(DanalornConfig.from_dict(danalorn_raw(width))),
            "basitar": model_figures(BasitarConfig.from_dict(dense_basitar_raw(width))),
            "qwen3": model_figures(Qwen3Config.from_dict(qwen3_raw(width, layers=6))),
            "kernels": kernel_figures(width, hbm_gbs),
        }
    return result


def main() -> int:
    parser = argparse.ArgumentParser(description=__doc__.splitlines()[0])
    parser.add_argument("--sizes", default="2048,4096")
    parser.add_argument("--hbm-gbs", type=float, default=6650.0)
    parser.add_argument("--alone", action="store_true", help="only launch the kernels a few times (for a profiler)")
    args = parser.parse_args()
    if args.alone:
        alone(int(args.sizes.split(",")[0]))
        return 0
    print(json.dumps(run([int(s) for s in args.sizes.split(",") if s], args.hbm_gbs)))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
