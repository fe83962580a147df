"""Prefill and decode throughput of Bidetar models at layer sizes of real models, beside Zupupel, Mezadra and Qwen3 of
equal width and depth, and the kernels that came with the design (or got a new form for it) alone, each next to the like
kernel of the closest model in the same harness.

    python bench.py --workload bidetar [--sizes 2048,4096]
    python -m rapid_llm_b200.ops.bidetar_compare [--sizes 2048,4096]
    python -m rapid_llm_b200.ops.bidetar_compare --alone --sizes 2048      # the kernels a few times each, for ncu

Random weights, bfloat16, one GPU.  A model of width ``W`` has four layers of which the middle two run twice (six layer
runs): ``W / 128`` heads of 128 over ``W / 512`` key/value heads, all 128 entries rotated with banded frequencies, chunks
of 512 positions, a feed-forward of ``4 W``.  Zupupel, Mezadra and Qwen3 beside it have six layers of the same width
(Qwen3's gated feed-forward has ``8 W / 3``, the same number of weights).  Prefill is one 2,048-token step (best of
three, CUDA events around the step function); decode is batch 8 behind 1,024-token prompts, replayed from the captured
graph (median of 32 steps).  Kernels are timed alone with CUDA events, L2 flushed between runs (a write of 256 MB), on one
2,048-token prompt and on 64 (products also on 8) single tokens behind 1,535 cached ones (the last of their chunk); ``frac`` is (bytes the kernel
must move) / time / measured copy bandwidth, ``tflops`` the products' arithmetic over the same time.
"""

from __future__ import annotations

import argparse
import json
import statistics
from types import SimpleNamespace

import torch

from .mezadra_compare import mezadra_raw
from .recurrent_compare import PREFILL, _events, model_figures, qwen3_raw
from .zupupel_compare import zupupel_raw

CHUNK = 512


def bidetar_raw(width: int) -> dict:
    heads = width // 128
    mixer = {"heads": heads, "kv_heads": max(heads // 4, 1), "dim": 128, "vdim": 128, "mask": {"size": CHUNK},
             "rot": {"dims": 128, "base": 5.0e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}},
             "scale": 128 ** -0.5}
    return {"architecture": "Bidetar", "vocab": 32000, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "residual_mult": 0.5, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "attention", "mixer": dict(mixer), "mlp": {"kind": "dense", "ff": 4 * width}} for _ in range(4)]}


def kernel_figures(width: int, hbm_gbs: float) -> dict:
    """The design's own kernels alone, and beside each the like kernel of the closest model, on a 2,048-token prompt and
    on single tokens."""
    import numpy as np

    from ..parts.attention import AttentionItems
    from ..parts.base import StepShape
    from . import gemm, kernels

    device = "cuda:0"
    heads, kv_heads, d, ff = width // 128, max(width // 512, 1), 128, 4 * width
    glu = (8 * width // 3 + 255) // 256 * 256
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
    workspace = SimpleNamespace(get=lambda name, rows, cols, dtype, min_rows=None: torch.empty(rows, cols, dtype=dtype, device=device))
    page, context = 16, 1535       # the single tokens are the last of a chunk: they see as many keys as the window lets them
    mix_rows = (heads + kv_heads) * d + -(-heads // 8) * 8
    first, last = bf(ff + mix_rows, width) / width ** 0.5, bf(width, ff + heads * d) / width ** 0.5
    first_bias, out_bias = f32(ff + mix_rows), f32(width)
    gate_up, down = bf(2 * glu, width) / width ** 0.5, bf(width, glu) / width ** 0.5
    for tokens, entries in ((PREFILL, 1), (64, 64), (8, 8)):
        # -- the stacked products, beside Qwen3's gate/up and down products
        x = bf(tokens, width)
        wide = torch.empty(tokens, ff + mix_rows, dtype=torch.bfloat16, device=device)
        timed("first product: feed-forward and mixer stacked, bias, squared relu", tokens, entries,
              first.numel() * 2 + x.numel() * 2 + wide.numel() * 2,
              lambda: gemm.linear(x, first, wide, fault, bias=first_bias, relu2_columns=ff), flops=2.0 * tokens * first.numel())
        act = torch.empty(tokens, glu, dtype=torch.bfloat16, device=device)
        timed("gate/up product with SiLU (like kernel)", tokens, entries, gate_up.numel() * 2 + x.numel() * 2 + act.numel() * 2,
              lambda: gemm.gated_linear(x, gate_up, act, workspace, fault), flops=2.0 * tokens * gate_up.numel())
        ready, result = wide[:, : last.shape[1]].copy_(bf(tokens, last.shape[1])), torch.empty(tokens, width, dtype=torch.bfloat16, device=device)
        stream, weight = f32(tokens, width), f32(width)
        offer = gemm.FollowingNorm(stream, weight, 1e-6, workspace, 0.5) if tokens <= 64 else None
        timed("last product: feed-forward and mixer side by side, bias" + (", sum and norm riding" if offer else ""), tokens, entries,
              last.numel() * 2 + ready.numel() * 2 + result.numel() * (10 if offer else 2),
              lambda: gemm.linear(ready, last, result, fault, then_norm=offer, bias=out_bias), flops=2.0 * tokens * last.numel())
        plain_offer = gemm.FollowingNorm(stream, weight, 1e-6, workspace) if tokens <= 64 else None
        timed("down product" + (", sum and norm riding" if offer else "") + " (like kernel)", tokens, entries,
              down.numel() * 2 + act.numel() * 2 + result.numel() * (10 if offer else 2),
              lambda: gemm.linear(act, down, result, fault, then_norm=plain_offer), flops=2.0 * tokens * down.numel())
        if tokens == 8:
            continue
        # -- the square of relu by itself (behind the library's product), beside SiLU times up
        timed("relu_squared, in place", tokens, entries, tokens * ff * 4, lambda: kernels.relu_squared(wide[:, :ff], wide[:, :ff]))
        pair = bf(tokens, 2 * glu)
        timed("silu_mul (like kernel)", tokens, entries, tokens * glu * 6, lambda: kernels.silu_mul(pair, act))
        # -- the sum with the stream and the norm, weighed and not
        timed("add_rmsnorm, weighed sum", tokens, entries, tokens * width * 12,
              lambda: kernels.add_rmsnorm(x, stream, weight, result, 1e-6, mode=1, write_residual=True, x_scale=0.5))
        timed("add_rmsnorm (like kernel)", tokens, entries, tokens * width * 12,
              lambda: kernels.add_rmsnorm(x, stream, weight, result, 1e-6, mode=1, write_residual=True))
        # -- norm over the whole projection, rotation of neighbours and cache write with the keys as values
        per, start = tokens // entries, 0 if entries == 1 else context
        pages_per = -(-(start + per) // page)
        cache = torch.zeros(entries * pages_per + 1, 2, kv_heads, page, d, dtype=torch.bfloat16, device=device)
        cache.normal_()
        table = (1 + torch.arange(entries * pages_per, dtype=torch.int32, device=device)).view(entries, pages_per)
        positions = (start + torch.arange(per, dtype=torch.int32, device=device)).repeat(entries)
        slots = torch.arange(entries, dtype=torch.int32, device=device)
        slot_of = slots.repeat_interleave(per)
        dest = (table[slot_of.long(), (positions // page).long()] * page + positions % page).to(torch.int32)
        q = torch.empty(tokens, heads * d, dtype=torch.bfloat16, device=device)
        q_weight, k_weight, freq = f32(heads * d), f32(kv_heads * d), torch.rand(64, device=device)
        shape = dict(num_heads=heads, num_kv_heads=kv_heads, head_dim=d, q_weight=q_weight, k_weight=k_weight, q_count=heads * d,
                     k_count=kv_heads * d, inv_freq=freq, positions=positions, eps=1e-6, fault=fault, kv_dest=dest, cache=cache,
                     page_size=page)
        mixer_columns = wide[:, ff:]
        timed("row_norm_rope_write, neighbours, values from keys", tokens, entries, tokens * (2 * heads + 3 * kv_heads) * d * 2,
              lambda: kernels.row_norm_rope_write(mixer_columns, q, neighbours=True, values_are_keys=True, **shape))
        qkv = bf(tokens, (heads + 2 * kv_heads) * d)
        timed("row_norm_rope_write, halves (like kernel)", tokens, entries, tokens * (heads + 2 * kv_heads) * d * 4,
              lambda: kernels.row_norm_rope_write(qkv, q, **shape))
        # -- attention: chunks, a sink and the gate; beside a window of the same size, and beside all keys
        cu = torch.arange(0, tokens + 1, per, dtype=torch.int32, device=device)
        starts = torch.full((entries,), start, dtype=torch.int32, device=device)
        sink, gate, attended = f32(heads), bf(tokens, heads), torch.empty_like(q)
        step = StepShape(lengths=np.full(entries, per, dtype=np.int32), starts=np.full(entries, start, dtype=np.int32),
                         decode_only=per == 1, page_size=page)
        every = start + np.arange(per)
        for label, window, chunk, extras in (
                ("attention, chunks, sink, gate", 0, CHUNK, {"sink": sink, "gate": gate}),
                ("attention, window of the same size (like kernel)", CHUNK, 0, {}), ("attention, all keys (like kernel)", 0, 0, {})):
            plan = AttentionItems(heads // kv_heads, kv_heads, d, chunk=chunk).plan(step)
            chunk_items, decode_items = (torch.from_numpy(plan[name]).to(device) for name in ("chunk_items", "decode_items"))
            splits = plan["splits"]
            rows = tokens * heads * splits
            part_out = torch.empty(rows, d, device=device) if splits > 1 else None
            part_lse = torch.empty(rows, 1, device=device) if splits > 1 else None
            seen = every % chunk + 1 if chunk else np.minimum(every + 1, window) if window else every + 1
            read = int(min(start + per, chunk and every[-1] % chunk + 1 or window or start + per)) if per == 1 else start + per
            timed(label, tokens, entries, entries * read * kv_heads * d * 4 + tokens * heads * d * 4,
                  lambda: kernels.attention_mma(
                      q, cache, attended, chunk_items=chunk_items, decode_items=decode_items, splits=splits, part_out=part_out,
                      part_lse=part_lse, cu_seqlens=cu, entry_start=starts, entry_slot=slots, block_table=table, num_heads=heads,
                      num_kv_heads=kv_heads, head_dim=d, window=window, chunk=chunk, scale=d ** -0.5, fault=fault,
                      decode_rows=plan["decode_rows"], chunk_rows=plan["chunk_rows"], decode_splits=plan["decode_splits"], **extras),
                  flops=4.0 * entries * int(seen.sum()) * heads * d)
    assert int(fault.item()) == 0, "a kernel reported a fault"
    return out


def alone(width: int = 2048) -> None:
    """Every kernel of :func:`kernel_figures` a few times and nothing else: the case a profiler captures, picking its
    kernel by name."""
    kernel_figures(width, 6650.0)
    torch.cuda.synchronize()


def run(sizes: list[int], hbm_gbs: float) -> dict:
    from ..config import BidetarConfig, MezadraConfig, Qwen3Config, ZupupelConfig

    result = {"workload": "bidetar beside zupupel, mezadra and qwen3, equal sizes", "dtype": "bf16", "data": "synthetic",
              "prefill_tokens": PREFILL, "decode_batch": 8, "decode_context": 1024, "sizes": {}}
    for width in sizes:
        result["sizes"][str(width)] = {
            "bidetar": model_figures(BidetarConfig.from_dict(bidetar_raw(width))),
            "zupupel": model_figures(ZupupelConfig.from_dict(zupupel_raw(width))),
            "mezadra": model_figures(MezadraConfig.from_dict(mezadra_raw(width))),
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
