"""The kernels that came with the Danalorn decoder, or got a new form for it, one by one, against plain PyTorch."""

from __future__ import annotations

import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def _word():
    return torch.zeros(1, dtype=torch.int32, device=DEVICE)


def _tolerance(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.6e-2, atol=1.6e-2)


# ------------------------------------------------------------------------------------ embedding -- #
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("scale", [1.0, 7.5])
def test_a_scaled_token_row_and_a_pair_row_without_positions(scale, dtype):
    """Entries at position 0 take the last row, others the token their slot kept; multipliers whose products pass 32 bits."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(1)
    vocab, buckets, hidden, mul_prev, mul_cur = 50, 31, 40, 1_000_000_007, 998_244_353
    lengths, starts, slots = [3, 1, 5], [0, 2_000_000, 7], [2, 0, 3]
    ids = torch.randint(0, vocab, (sum(lengths),), generator=g)
    kept = torch.randint(0, vocab, (4, 1), generator=g)
    table, pair = torch.randn(vocab, hidden, generator=g).to(dtype), torch.randn(buckets + 1, hidden, generator=g).to(dtype)
    rows, at = [], 0
    for length, start, slot in zip(lengths, starts, slots):
        before = int(kept[slot])
        for place in range(length):
            token = int(ids[at])
            row = buckets if start + place == 0 else (before * mul_prev + token * mul_cur) % buckets
            rows.append(scale * table[token].float() + pair[row].float())
            before, at = token, at + 1
    want = torch.stack(rows)
    positions = torch.cat([start + torch.arange(length) for length, start in zip(lengths, starts)]).to(torch.int32)
    batch = SimpleNamespace(token_ids=ids.to(torch.int32).to(DEVICE), feedback=None, positions=positions.to(DEVICE),
                            cu_seqlens=torch.tensor([0, 3, 4, 9], dtype=torch.int32, device=DEVICE),
                            entry_slot=torch.tensor(slots, dtype=torch.int32, device=DEVICE), num_entries=3, fault=_word())
    out = torch.empty(9, hidden, dtype=dtype, device=DEVICE)
    stream = torch.empty(9, hidden, device=DEVICE)
    last = kept.to(torch.int32).to(DEVICE)
    kernels.embedding_sum(out, stream, table.to(DEVICE), pair.to(DEVICE), None, batch, last, mul_prev=mul_prev, mul_cur=mul_cur, scale=scale)
    assert int(batch.fault.item()) == 0
    torch.testing.assert_close(stream.cpu(), want, rtol=1e-6, atol=1e-6)
    torch.testing.assert_close(out.cpu().float(), want.to(dtype).float(), **_tolerance(dtype))
    assert last.flatten().tolist() == [int(ids[3]), int(kept[1]), int(ids[2]), int(ids[8])]


# --------------------------------------------------------------------------------- query and key -- #
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 9, 700])
@pytest.mark.parametrize("hq,hkv,d,true_d,rotary,temperature", [
    (6, 2, 16, 10, 0, (0.5, 7.0)), (4, 2, 32, 32, 0, (0.3, 128.0)), (8, 8, 64, 60, 0, None), (5, 5, 96, 90, 0, (1.5, 1.0)), (12, 4, 128, 128, 0, (0.5, 64.0)),
    (12, 4, 128, 128, 128, (0.5, 64.0)), (2, 1, 256, 200, 0, (0.25, 33.0)), (12, 4, 128, 128, 128, None), (4, 2, 96, 96, 96, None), (3, 3, 48, 40, 16, (0.7, 10.0))])
def test_norm_per_head_without_rotation_and_with_a_temperature(hq, hkv, d, true_d, rotary, temperature, tokens, dtype):
    """q, k and v as the first columns of wider rows; a head's padding holds zeros; the temperature steps at multiples of
    its stretch, whatever the kernel's form (registers, pairs of heads, through shared memory)."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(hq * d + tokens)
    page_size, extra = 16, 24
    pages = -(-tokens // page_size) + 2
    heads = hq + 2 * hkv
    inner = torch.randn(tokens, heads, d, generator=g)
    inner[:, :, true_d:] = 0.0
    wide = torch.full((tokens, heads * d + extra), float("nan"))
    wide[:, : heads * d] = inner.view(tokens, -1)
    wide = wide.to(dtype).to(DEVICE)
    q_weight, k_weight = (torch.cat([1 + 0.3 * torch.randn(true_d, generator=g), torch.zeros(d - true_d)]) for _ in range(2))
    positions = torch.randint(0, 2000, (tokens,), generator=g).to(torch.int32)
    if temperature:
        edges = [int(temperature[1]) * n + off for n in (1, 2, 9) for off in (-2, -1, 0)]
        for place, position in enumerate(edges[:tokens]):
            positions[place] = max(position, 0)
    angles = torch.outer(torch.arange(2304, dtype=torch.float32), 50.0 ** (-torch.arange(0, rotary, 2, dtype=torch.float32) / max(rotary, 1)))
    cos, sin = torch.cos(angles).contiguous(), torch.sin(angles).contiguous()
    dest = (torch.randperm(page_size * (pages - 1), generator=g)[:tokens] + page_size).to(torch.int32)
    cache = torch.zeros(pages, 2, hkv, page_size, d, dtype=dtype, device=DEVICE)
    q_out, fault = torch.empty(tokens, hq * d, dtype=dtype, device=DEVICE), _word()
    kernels.qk_norm_rope_write(wide, q_out, num_heads=hq, num_kv_heads=hkv, head_dim=d, rotary_dim=rotary, cos=cos.to(DEVICE), sin=sin.to(DEVICE),
                               positions=positions.to(DEVICE), eps=1e-5, fault=fault, q_weight=q_weight.to(DEVICE), k_weight=k_weight.to(DEVICE),
                               kv_dest=dest.to(DEVICE), cache=cache, page_size=page_size, norm_size=true_d, temperature=temperature)
    assert int(fault.item()) == 0
    rows = inner.to(dtype).double()

    def finished(part, weight):
        out = part * torch.rsqrt((part * part).sum(-1, keepdim=True) / true_d + 1e-5) * weight.double()
        if rotary:
            c, s = (t[positions.long()].double()[:, None] for t in (cos, sin))
            u, v = out[..., : rotary // 2].clone(), out[..., rotary // 2 : rotary].clone()
            out[..., : rotary // 2], out[..., rotary // 2 : rotary] = u * c - v * s, v * c + u * s
        return out

    q = finished(rows[:, :hq], q_weight)
    if temperature:
        coef, every = temperature
        q = q * torch.tensor([1.0 + coef * math.log((int(p) + 1) // int(every) + 1) for p in positions]).double()[:, None, None]
    bound = dict(rtol=2e-5, atol=5e-5) if dtype == torch.float32 else dict(rtol=1.2e-2, atol=1.2e-2)
    torch.testing.assert_close(q_out.cpu().double().view(tokens, hq, d), q, **bound)
    stored = cache.cpu().double().permute(0, 3, 1, 2, 4).reshape(-1, 2, hkv, d)[dest.long()]
    torch.testing.assert_close(stored[:, 0], finished(rows[:, hq : hq + hkv], k_weight), **bound)
    assert torch.equal(stored[:, 1], rows[:, hq + hkv :])


@pytest.mark.parametrize("rotary", [0, 96])
def test_every_head_of_an_odd_multiple_of_32_is_written_at_many_tokens(rotary):
    """Heads of 96 have no form in registers: at tens of thousands of heads a step each still gets a warp of its own."""
    from rapid_llm_b200.ops import kernels

    tokens, hq, hkv, d, page_size = 10_000, 6, 1, 96, 16
    g = torch.Generator(device=DEVICE).manual_seed(2)
    qkv = torch.randn(tokens, (hq + 2 * hkv) * d, generator=g, device=DEVICE).to(torch.bfloat16)
    table = torch.zeros(64, rotary // 2, device=DEVICE)
    cache = torch.zeros(tokens // page_size + 1, 2, hkv, page_size, d, dtype=torch.bfloat16, device=DEVICE)
    q_out, fault = torch.full((tokens, hq * d), 7.0, dtype=torch.bfloat16, device=DEVICE), _word()
    kernels.qk_norm_rope_write(qkv, q_out, num_heads=hq, num_kv_heads=hkv, head_dim=d, rotary_dim=rotary, cos=table + 1.0, sin=table,
                               positions=torch.arange(tokens, dtype=torch.int32, device=DEVICE) % 64, eps=1e-6, fault=fault,
                               kv_dest=page_size + torch.arange(tokens, dtype=torch.int32, device=DEVICE), cache=cache, page_size=page_size)
    assert int(fault.item()) == 0
    assert torch.equal(q_out, qkv[:, : hq * d])
    stored = cache.permute(0, 3, 1, 2, 4).reshape(-1, 2 * d)[page_size : page_size + tokens]
    assert torch.equal(stored, qkv[:, hq * d :])


# -------------------------------------------------------------------------------------- latents -- #
@pytest.mark.parametrize("dtype", DTYPES)
def test_a_query_latent_alone_is_normed_without_a_cache(dtype):
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(3)
    down = torch.randn(19, 24, generator=g).to(dtype).to(DEVICE)
    weight = (1 + 0.2 * torch.randn(21, generator=g)).to(DEVICE)
    out, fault = torch.empty(19, 21, dtype=dtype, device=DEVICE), _word()
    kernels.latent_norm_write(down, q_col0=0, q_rank=21, c_col0=24, kv_rank=50, rot=6, q_weight=weight, c_weight=None, eps=1e-5, q_out=out,
                              cache=None, kv_dest=None, positions=torch.zeros(19, dtype=torch.int32, device=DEVICE), freq=torch.ones(3, device=DEVICE),
                              magnitude=1.0, layout=kernels.ROTATE_NEIGHBOURS, fault=fault)
    assert int(fault.item()) == 0
    x = down.float()[:, :21]
    torch.testing.assert_close(out.float(), (x * torch.rsqrt((x * x).mean(-1, keepdim=True) + 1e-5) * weight).to(dtype).float(), **_tolerance(dtype))


# --------------------------------------------------------------------------------------- decays -- #
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 7, 8, 130])
@pytest.mark.parametrize("copied,channels,rank,tau", [(36, 24, 5, 6.0), (33, 130, 1, 1.0), (512, 256, 32, 16.0), (40, 129, 64, 2.5), (1300, 7, 41, 0.5), (8, 300, 16, 16.0)])
def test_decays_from_a_low_rank_product(copied, channels, rank, tau, tokens, dtype):
    """``sigmoid(z) ** (1 / tau)`` in float32 for z from far below to far above zero, columns copied as float32, everything
    between the two left alone; a row's result is the same whatever rows are beside it."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(copied + rank)
    low_col0 = -(-copied // 8) * 8 + 16
    buffer = torch.randn(tokens, low_col0 + -(-rank // 8) * 8, generator=g).to(dtype).to(DEVICE)
    weight = (torch.randn(channels, rank, generator=g) * 2 / math.sqrt(rank)).to(dtype).to(DEVICE)
    bias = (torch.randn(channels, generator=g) * 6).to(DEVICE)
    rows, decay = torch.full((tokens, copied), 7.0, device=DEVICE), torch.full((tokens, channels), 7.0, device=DEVICE)
    kernels.low_rank_decay(buffer[:, :copied], buffer[:, low_col0 : low_col0 + rank], weight, bias, tau, rows, decay)
    assert torch.equal(rows, buffer[:, :copied].float())
    z = buffer[:, low_col0 : low_col0 + rank].double() @ weight.double().T + bias.double()
    torch.testing.assert_close(decay.double(), torch.exp(torch.nn.functional.logsigmoid(z) / tau), rtol=3e-6, atol=1e-6)
    again_rows, again = torch.empty(1, copied, device=DEVICE), torch.empty(1, channels, device=DEVICE)
    one = buffer[-1:].clone()
    kernels.low_rank_decay(one[:, :copied], one[:, low_col0 : low_col0 + rank], weight, bias, tau, again_rows, again)
    assert torch.equal(again[0], decay[-1])


# ------------------------------------------------------------------------------------- attention -- #
def _case(dtype, hq, hkv, d, page, lengths, new, seed, planes=2):
    """A paged cache in which request r has ``lengths[r]`` tokens of which the last ``new[r]`` are this step's; page ids are
    shuffled, unused places hold numbers that must not count."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-length // page) for length in lengths]
    order = (torch.randperm(sum(per), generator=g) + 1).tolist()
    cache = torch.full((sum(per) + 1, planes, hkv, page, d), 50.0, dtype=dtype)
    table = torch.zeros(len(lengths) + 1, max(per) + 1, dtype=torch.int32)
    slots = torch.randperm(len(lengths), generator=g).tolist()
    out = {"keys": [], "values": [], "queries": [], "positions": [], "token_slot": []}
    for length, fresh, count, slot in zip(lengths, new, per, slots):
        pages = [order.pop() for _ in range(count)]
        table[slot, :count] = torch.tensor(pages, dtype=torch.int32)
        rows = torch.randn(length, planes, hkv, d, generator=g).to(dtype)
        for j in range(length):
            cache[pages[j // page], :, :, j % page] = rows[j]
        out["keys"].append(rows[:, 0].double())
        out["values"].append(rows[:, -1].double())
        out["queries"].append((torch.randn(fresh, hq, d, generator=g)).to(dtype))
        out["positions"] += list(range(length - fresh, length))
        out["token_slot"] += [slot] * fresh
    return {**out, "q": torch.cat(out["queries"]).reshape(-1, hq * d).to(DEVICE), "cache": cache.to(DEVICE), "table": table.to(DEVICE),
            "slots": torch.tensor(slots, dtype=torch.int32, device=DEVICE), "positions": torch.tensor(out["positions"], dtype=torch.int32, device=DEVICE),
            "token_slot": torch.tensor(out["token_slot"], dtype=torch.int32, device=DEVICE)}


def _plain(case, hq, hkv, lengths, new, scale, window=0, sink=None, slopes=None):
    rows = []
    for key, value, query, length, fresh in zip(case["keys"], case["values"], case["queries"], lengths, new):
        for offset in range(fresh):
            i = length - fresh + offset
            first = max(0, i - window + 1) if window else 0
            k, v = (t[first : i + 1].repeat_interleave(hq // hkv, dim=1) for t in (key, value))
            scores = torch.einsum("hd,jhd->hj", query[offset].double(), k) * scale
            if slopes is not None:
                scores = scores - slopes.double().cpu()[:, None] * (i - torch.arange(first, i + 1)).double()[None]
            if sink is not None:
                scores = torch.cat([scores, sink.double().cpu()[:, None]], dim=1)
            weights = torch.softmax(scores, dim=1)[:, : k.shape[0]]
            rows.append(torch.einsum("hj,jhd->hd", weights, v).reshape(-1))
    return torch.stack(rows).float()


def _slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], device=DEVICE)


def _tiles(case, hq, hkv, d, page, lengths, new, out, *, window=0, sink=None, slopes=None, splits=None, decode_kernel="auto", tensor_core=True):
    from rapid_llm_b200.ops import kernels
    from rapid_llm_b200.parts.attention import AttentionItems
    from rapid_llm_b200.parts.base import StepShape

    starts = np.asarray(lengths, np.int32) - np.asarray(new, np.int32)
    planner = AttentionItems(hq // hkv, hkv, d, tensor_core=tensor_core, window=window)
    plan = planner.plan(StepShape(np.asarray(new, np.int32), starts, decode_only=max(new) == 1, page_size=page))
    if splits is not None and splits != plan["splits"]:
        def respread(items):
            base = items[items[:, 2] == 0]
            again = np.repeat(base, splits, axis=0)
            again[:, 2] = np.tile(np.arange(splits, dtype=np.int32), len(base))
            return again
        assert plan["chunk_rows"] == kernels.CHUNK_TILE_ROWS or not len(plan["chunk_items"])
        plan = dict(plan, chunk_items=respread(plan["chunk_items"]), decode_items=respread(plan["decode_items"]), splits=splits, decode_splits=splits)
    tokens, count = case["q"].shape[0], plan["splits"]
    part_out = torch.full((tokens * hq * count, d), float("nan"), device=DEVICE) if count > 1 else None
    part_lse = torch.full((tokens * hq * count,), float("nan"), device=DEVICE) if count > 1 else None
    fault = _word()
    kernels.attention_mma(
        case["q"], case["cache"], out, chunk_items=torch.from_numpy(plan["chunk_items"]).to(DEVICE), decode_items=torch.from_numpy(plan["decode_items"]).to(DEVICE),
        splits=count, part_out=part_out, part_lse=part_lse, cu_seqlens=torch.tensor([0] + list(np.cumsum(new)), dtype=torch.int32, device=DEVICE),
        entry_start=torch.from_numpy(starts).to(DEVICE), entry_slot=case["slots"], block_table=case["table"], num_heads=hq, num_kv_heads=hkv, head_dim=d,
        window=window, scale=d ** -0.5, fault=fault, decode_kernel=decode_kernel, decode_rows=plan["decode_rows"], chunk_rows=plan["chunk_rows"],
        decode_splits=plan["decode_splits"], sink=sink, slopes=slopes)
    assert int(fault.item()) == 0
    return plan


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hq,hkv,d,page,planes,window", [(6, 2, 16, 8, 2, 0), (3, 3, 48, 16, 2, 0), (8, 1, 128, 16, 2, 70), (5, 1, 272, 16, 1, 31), (4, 1, 80, 4, 1, 0)])
def test_one_warp_per_row_attention_with_slopes_and_a_sink(hq, hkv, d, page, planes, window, dtype):
    from rapid_llm_b200.ops import kernels

    lengths, new = [1, 15, 24, 25, 129, 200], [1, 15, 1, 2, 129, 33]
    case = _case(dtype, hq, hkv, d, page, lengths, new, seed=d + page, planes=planes)
    sink, slopes, fault = torch.zeros(hq, device=DEVICE), _slopes(hq), _word()
    out = torch.empty_like(case["q"])
    kernels.attention_generic(case["q"], case["cache"], out, positions=case["positions"], token_slot=case["token_slot"], block_table=case["table"],
                              num_heads=hq, num_kv_heads=hkv, head_dim=d, window=window, scale=d ** -0.5, fault=fault, sink=sink, slopes=slopes)
    assert int(fault.item()) == 0
    bound = {"rtol": 1e-4, "atol": 2e-5} if dtype == torch.float32 else {"rtol": 3e-2, "atol": 8e-3}
    torch.testing.assert_close(out.float().cpu(), _plain(case, hq, hkv, lengths, new, d ** -0.5, window, sink, slopes), **bound)


@pytest.mark.parametrize("fixed_sink", [True, False])
@pytest.mark.parametrize("hq,hkv,d,page,splits", [
    (8, 2, 128, 16, None), (12, 3, 128, 8, None), (4, 4, 128, 64, None), (5, 5, 128, 16, None), (6, 1, 32, 8, None), (6, 1, 32, 8, 3), (7, 7, 48, 4, 2),
    (4, 2, 64, 16, None), (3, 1, 256, 64, None), (40, 2, 64, 16, 4)])
def test_prompt_and_decode_tiles_with_slopes(hq, hkv, d, page, splits, fixed_sink):
    """Portions of prompts beside single tokens: the tcgen05 tiles at heads of 128, the mma.sync tiles elsewhere, whole and
    with split key ranges; the first head's slope leaves a handful of keys, the last one's reaches hundreds back."""
    lengths, new = [1, 15, 16, 17, 129, 200, 64, 700, 333, 301], [1, 15, 1, 2, 129, 1, 33, 1, 170, 1]
    case = _case(torch.bfloat16, hq, hkv, d, page, lengths, new, seed=d + page)
    sink = torch.zeros(hq, device=DEVICE) if fixed_sink else None
    out = torch.full_like(case["q"], 7.0)
    plan = _tiles(case, hq, hkv, d, page, lengths, new, out, sink=sink, slopes=_slopes(hq), splits=splits)
    assert plan["chunk_rows"] == (256 if d == 128 else 64)
    want = _plain(case, hq, hkv, lengths, new, d ** -0.5, 0, sink, _slopes(hq))
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=8e-3)


@pytest.mark.parametrize("decode_kernel", ["auto", "mma", "deep", "shallow"])
@pytest.mark.parametrize("hq,hkv,page,splits,lengths", [
    (32, 8, 16, None, [1, 5, 128, 513, 1000, 257, 2049]), (8, 2, 16, 3, [700, 701, 1]), (40, 2, 64, 2, [400, 90]), (8, 1, 16, 10, [5000]),
    (4, 4, 8, 1, [131, 260, 130]), (16, 16, 16, None, [900, 3])])
def test_single_tokens_on_the_decode_tiles_with_slopes(hq, hkv, page, splits, lengths, decode_kernel):
    d, new = 128, [1] * len(lengths)
    case = _case(torch.bfloat16, hq, hkv, d, page, lengths, new, seed=page + hq)
    sink, out = torch.zeros(hq, device=DEVICE), torch.full_like(case["q"], 7.0)
    _tiles(case, hq, hkv, d, page, lengths, new, out, sink=sink, slopes=_slopes(hq), splits=splits, decode_kernel=decode_kernel)
    want = _plain(case, hq, hkv, lengths, new, d ** -0.5, 0, sink, _slopes(hq))
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=8e-3)


@pytest.mark.parametrize("hq,d,page,window,splits", [(6, 128, 16, 100, None), (6, 128, 16, 100, 3), (16, 256, 16, 65, None), (3, 48, 8, 1, None), (9, 32, 4, 64, 2), (40, 64, 16, 200, None),
                                                     (5, 128, 16, 0, None)])
def test_tiles_over_one_plane_with_a_window_and_a_sink(hq, d, page, window, splits):
    """Rows that are keys and values at once, shared by all heads: windows that begin inside, on and behind a block of keys
    and a page, in portions and single tokens, with a sink a head."""
    lengths, new = [1, 15, 16, 17, 129, 200, 64, 700, 333, 301], [1, 15, 1, 2, 129, 1, 33, 1, 170, 1]
    case = _case(torch.bfloat16, hq, 1, d, page, lengths, new, seed=d + page, planes=1)
    sink = torch.linspace(-4.0, 3.0, hq, device=DEVICE)
    out = torch.full_like(case["q"], 7.0)
    _tiles(case, hq, 1, d, page, lengths, new, out, window=window, sink=sink, splits=splits, decode_kernel="mma", tensor_core=False)
    want = _plain(case, hq, 1, lengths, new, d ** -0.5, window, sink)
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=8e-3)
    lengths = [1, 99, 100, 101, 650, 64, 65]
    new = [1] * len(lengths)
    case = _case(torch.bfloat16, hq, 1, d, page, lengths, new, seed=d, planes=1)
    out = torch.full_like(case["q"], 7.0)
    _tiles(case, hq, 1, d, page, lengths, new, out, window=window, sink=sink, splits=splits, decode_kernel="mma", tensor_core=False)
    torch.testing.assert_close(out.float().cpu(), _plain(case, hq, 1, lengths, new, d ** -0.5, window, sink), rtol=3e-2, atol=8e-3)


def test_slopes_over_one_plane_are_refused_by_the_tiles():
    from rapid_llm_b200.ops import kernels

    case = _case(torch.bfloat16, 2, 1, 32, 8, [20], [20], seed=1, planes=1)
    with pytest.raises(kernels.KernelError, match="invalid value"):
        _tiles(case, 2, 1, 32, 8, [20], [20], torch.empty_like(case["q"]), slopes=_slopes(2), decode_kernel="mma", tensor_core=False)
    with pytest.raises(kernels.KernelError, match="slopes"):
        _tiles(case, 2, 1, 32, 8, [20], [20], torch.empty_like(case["q"]), slopes=_slopes(3), decode_kernel="mma", tensor_core=False)
