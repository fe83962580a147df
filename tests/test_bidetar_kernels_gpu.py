"""The kernels that came with the Bidetar decoder, or got a new form for it, one by one, against plain PyTorch."""

from __future__ import annotations

import gc

import numpy as np
import pytest
import torch

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"


def _word():
    return torch.zeros(1, dtype=torch.int32, device=DEVICE)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq,hkv,d,true_d,rotary,values_are_keys", [(4, 2, 16, 16, 8, True), (6, 3, 32, 20, 20, True), (3, 3, 16, 10, 6, True),
                                                                   (8, 1, 64, 64, 0, True), (5, 5, 48, 48, 48, False), (8, 2, 128, 128, 128, True)])
def test_neighbours_rotate_together_and_keys_are_values(hq, hkv, d, true_d, rotary, values_are_keys, dtype):
    """Norm over the whole projection (the mean over the TRUE entries), rotation of entries 2i and 2i + 1, q out, keys into
    their pages, and as values the k columns as they came; read from some columns of wider rows."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(hq * d)
    tokens, page_size, pages, before = 23, 8, 9, 40
    width = (hq + (1 if values_are_keys else 2) * hkv) * d
    inner = torch.randn(tokens, width, generator=g)
    inner.view(tokens, -1, d)[:, :, torch.arange(d) >= true_d] = 0.0          # a head's padding holds zeros
    wide = torch.full((tokens, before + width + 16), float("nan"))
    wide[:, before : before + width] = inner
    wide = wide.to(dtype).to(DEVICE)
    q_weight, k_weight = (1 + 0.3 * torch.randn(h * d, generator=g) for h in (hq, hkv))
    freq = (100.0 ** (-torch.arange(0, rotary, 2, dtype=torch.float64) / max(rotary, 1))).float() if rotary else None
    positions = torch.randint(0, 3000, (tokens,), generator=g).to(torch.int32)
    dest = torch.randperm(page_size * (pages - 1), generator=g)[:tokens].to(torch.int32) + page_size
    cache = torch.zeros(pages, 2, hkv, page_size, d, dtype=dtype, device=DEVICE)
    q_out, fault = torch.empty(tokens, hq * d, dtype=dtype, device=DEVICE), _word()
    kernels.row_norm_rope_write(wide[:, before:], q_out, num_heads=hq, num_kv_heads=hkv, head_dim=d, q_weight=q_weight.to(DEVICE),
                                k_weight=k_weight.to(DEVICE), q_count=hq * true_d, k_count=hkv * true_d,
                                inv_freq=None if freq is None else freq.to(DEVICE), positions=positions.to(DEVICE), eps=1e-5, fault=fault,
                                kv_dest=dest.to(DEVICE), cache=cache, page_size=page_size, neighbours=True, values_are_keys=values_are_keys)
    assert int(fault.item()) == 0
    rows = inner.to(dtype).double()

    def normed(part, weight, count, heads):
        scaled = (part * torch.rsqrt((part * part).sum(-1, keepdim=True) / count + 1e-5) * weight.double()).view(tokens, heads, d)
        if rotary:
            angle = (positions.float()[:, None] * freq[None, :]).double()      # the angle itself is a float32 product
            pairs = torch.view_as_complex(scaled[..., :rotary].reshape(tokens, heads, rotary // 2, 2).contiguous())
            turned = pairs * torch.polar(torch.ones_like(angle), angle)[:, None, :]
            scaled = torch.cat([torch.view_as_real(turned).reshape(tokens, heads, rotary), scaled[..., rotary:]], dim=-1)
        return scaled

    bound = {"rtol": 2e-5, "atol": 2e-5} if dtype == torch.float32 else {"rtol": 1e-2, "atol": 1e-2}
    q_width, k_width = hq * d, hkv * d
    want_q = normed(rows[:, :q_width], q_weight, hq * true_d, hq).reshape(tokens, -1).float()
    want_k = normed(rows[:, q_width : q_width + k_width], k_weight, hkv * true_d, hkv).float()
    want_v = rows[:, q_width : q_width + k_width] if values_are_keys else rows[:, q_width + k_width :]
    torch.testing.assert_close(q_out.float().cpu(), want_q, **bound)
    for t in range(tokens):
        page, offset = int(dest[t]) // page_size, int(dest[t]) % page_size
        torch.testing.assert_close(cache[page, 0, :, offset].float().cpu(), want_k[t], **bound)
        assert torch.equal(cache[page, 1, :, offset].double().cpu().reshape(-1), want_v[t].reshape(-1))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,stride,column", [(64, 64, 0), (40, 104, 24), (13, 30, 5)])
def test_the_square_of_relu_in_place_on_some_columns(width, stride, column, dtype):
    from rapid_llm_b200.ops import kernels

    base = torch.randn(37, stride, generator=torch.Generator().manual_seed(width)).to(dtype)
    rows = base.to(DEVICE)
    part = rows[:, column : column + width]
    kernels.relu_squared(part, part)
    want = base.clone()
    want[:, column : column + width] = (base[:, column : column + width].float().clamp(min=0) ** 2).to(dtype)
    assert torch.equal(rows.cpu(), want)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,before", [(48, 16), (13, 3)])
def test_a_gate_entry_by_entry_into_the_columns_beside_it(width, before, dtype):
    """The result goes to some columns of the rows that also hold the gate, as in a stack of products."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(width)
    rows = torch.randn(21, width, generator=g).to(dtype)
    base = torch.randn(21, before + 2 * width + 8, generator=g).to(dtype)
    wide = base.to(DEVICE)
    gate = wide[:, before + width : before + 2 * width]
    kernels.sigmoid_gate(rows.to(DEVICE), gate, wide[:, before : before + width])
    want = rows.float() * torch.sigmoid(base[:, before + width : before + 2 * width].float())
    bound = {"rtol": 1e-5, "atol": 1e-6} if dtype == torch.float32 else {"rtol": 1e-2, "atol": 1e-2}
    torch.testing.assert_close(wide[:, before : before + width].float().cpu(), want, **bound)
    assert torch.equal(wide[:, :before].cpu(), base[:, :before]) and torch.equal(wide[:, before + width :].cpu(), base[:, before + width :])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hidden", [64, 50, 1032])
def test_what_joins_the_stream_is_weighed(hidden, dtype):
    """``residual <- residual + m * x`` in float32, and the norm of it; every row, and picked rows without storing."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(hidden)
    x = torch.randn(9, hidden, generator=g).to(dtype).to(DEVICE)
    stream, weight = torch.randn(9, hidden, generator=g).to(DEVICE), (1 + 0.2 * torch.randn(hidden, generator=g)).to(DEVICE)
    before, out = stream.clone(), torch.empty(9, hidden, dtype=dtype, device=DEVICE)
    kernels.add_rmsnorm(x, stream, weight, out, 1e-5, mode=1, write_residual=True, x_scale=0.37)
    total = before.double() + 0.37 * x.double()
    torch.testing.assert_close(stream.double(), total, rtol=1e-6, atol=1e-6)
    normed = total * torch.rsqrt(total.pow(2).mean(-1, keepdim=True) + 1e-5) * weight.double()
    bound = {"rtol": 1e-5, "atol": 1e-5} if dtype == torch.float32 else {"rtol": 1e-2, "atol": 1e-2}
    torch.testing.assert_close(out.double(), normed, **bound)
    picked = torch.tensor([7, 0, 7], dtype=torch.int32, device=DEVICE)
    some, kept = torch.empty(3, hidden, dtype=dtype, device=DEVICE), before.clone()
    kernels.add_rmsnorm(x, kept, weight, some, 1e-5, mode=1, write_residual=False, row_index=picked, x_scale=0.37)
    assert torch.equal(kept, before) and torch.equal(some, out[picked.long()])


@pytest.mark.parametrize("tokens", [1, 7, 16, 40, 64, 200])
@pytest.mark.parametrize("n,k,split", [(1000, 256, 0), (520, 1024, 4), (130, 512, 1)])
def test_a_product_with_squared_columns_from_wider_rows(tokens, n, k, split):
    """The leading columns of a product pass the square of relu after the bias, the others do not, whatever tile or split
    they fall in; ``x`` is some columns of wider rows."""
    from rapid_llm_b200.ops import kernels

    g = torch.Generator().manual_seed(n + tokens)
    wide = torch.randn(tokens, k + 72, generator=g).to(torch.bfloat16).to(DEVICE)
    x = wide[:, 24 : 24 + k]
    w = (torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16).to(DEVICE)
    bias = torch.randn(n, generator=g).to(DEVICE)
    for columns in (0, 3, 128, n - 1, n):
        out = torch.full((tokens, n), float("nan"), dtype=torch.bfloat16, device=DEVICE)
        fault = _word()
        kernels.gemm_bf16(x, w, out, fault, bias=bias, relu2_columns=columns, k_split=split)
        want = x.double() @ w.double().T + bias.double()
        want[:, :columns] = want[:, :columns].clamp(min=0) ** 2
        assert int(fault.item()) == 0
        torch.testing.assert_close(out.double(), want, rtol=1e-2, atol=1e-2)


@pytest.mark.parametrize("tokens", [1, 8, 33, 64])
@pytest.mark.parametrize("split", [0, 1, 4])
def test_a_product_that_joins_the_stream_weighed(tokens, split):
    """The norm that rides on the product: residual + m * (product + bias) in float32, the sum times the norm's weight,
    its squares; from some columns of wider rows."""
    from rapid_llm_b200.ops import kernels

    n, k = 264, 768
    g = torch.Generator().manual_seed(tokens)
    x = torch.randn(tokens, k + 64, generator=g).to(torch.bfloat16).to(DEVICE)[:, :k]
    w = (torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16).to(DEVICE)
    bias, weight, stream = (torch.randn(*shape, generator=g).to(DEVICE) for shape in ((n,), (n,), (tokens, n)))
    before, out = stream.clone(), torch.empty(tokens, n, dtype=torch.bfloat16, device=DEVICE)
    sumsq, fault = torch.empty(tokens, kernels.gemm_bf16_sumsq_count(n), device=DEVICE), _word()
    kernels.gemm_bf16(x, w, out, fault, bias=bias, residual=stream, norm_weight=weight, sumsq_out=sumsq, residual_scale=-0.4, k_split=split)
    assert int(fault.item()) == 0
    want = before.double() - 0.4 * (x.double() @ w.double().T + bias.double())
    torch.testing.assert_close(stream.double(), want, rtol=1e-5, atol=1e-5)
    torch.testing.assert_close(out.double(), want * weight.double(), rtol=1e-2, atol=1e-2)
    torch.testing.assert_close(sumsq.double().sum(-1), want.pow(2).sum(-1), rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("tokens", [5, 100])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_linear_squares_columns_on_every_path(tokens, dtype):
    """The tensor-core product (small steps), the library's (large ones), an inner size that neither TMA takes, and the
    32-bit product give the same thing."""
    from rapid_llm_b200.ops import gemm, kernels

    for k in (64, 50):
        g = torch.Generator().manual_seed(k)
        x = torch.randn(tokens, k, generator=g).to(dtype).to(DEVICE)
        w, bias = (torch.randn(96, k, generator=g) / k ** 0.5).to(dtype).to(DEVICE), torch.randn(96, generator=g).to(torch.bfloat16).float().to(DEVICE)
        out = torch.empty(tokens, 96, dtype=dtype, device=DEVICE)
        gemm.linear(x, w, out, _word(), bias=bias, relu2_columns=40)
        want = x.double() @ w.double().T + bias.double()
        want[:, :40] = want[:, :40].clamp(min=0) ** 2
        bound = {"rtol": 1e-5, "atol": 1e-5} if dtype == torch.float32 else {"rtol": 2e-2, "atol": 2e-2}
        torch.testing.assert_close(out.double(), want, **bound)
    offer = gemm.FollowingNorm(torch.zeros(tokens, 96, device=DEVICE), torch.ones(96, device=DEVICE), 1e-5, None)
    with pytest.raises(kernels.KernelError, match="activation"):
        gemm.linear(x, w, out, _word(), bias=bias, relu2_columns=40, then_norm=offer)


def test_a_bias_of_the_librarys_product_is_the_vector_given():
    """A vector that takes over a freed one's address, and one changed in place, are not served by the old one's copy."""
    from rapid_llm_b200.ops import gemm

    x = torch.zeros(100, 64, dtype=torch.bfloat16, device=DEVICE)
    w, out = torch.zeros(32, 64, dtype=torch.bfloat16, device=DEVICE), torch.empty(100, 32, dtype=torch.bfloat16, device=DEVICE)
    addresses = set()
    for value in (1.0, 2.0, 3.0):
        bias = torch.full((32,), value, device=DEVICE)
        addresses.add(bias.data_ptr())
        assert float(gemm.linear(x, w, out, _word(), bias=bias).float().mean()) == value
        bias.add_(0.5)
        assert float(gemm.linear(x, w, out, _word(), bias=bias).float().mean()) == value + 0.5
        del bias
        gc.collect()
    assert len(addresses) < 3, "the allocator handed out fresh addresses: the test shows nothing"


# -------------------------------------------------------------------------------------------- attention -- #
def _case(dtype, hq, hkv, d, page, lengths, new, seed):
    """Requests of given lengths on shuffled pages; the last ``new`` positions of each are this step's queries."""
    g = torch.Generator().manual_seed(seed)
    counts = [-(-length // page) for length in lengths]
    order = (torch.randperm(sum(counts), generator=g) + 1).tolist()
    table = torch.zeros(len(lengths) + 1, max(counts), dtype=torch.int32)
    slots = torch.randperm(len(lengths) + 1, generator=g)[: len(lengths)].tolist()
    cache = torch.randn(sum(counts) + 1, 2, hkv, page, d, generator=g).to(dtype)
    keys, values, queries, positions, token_slot = [], [], [], [], []
    for length, count, slot, fresh in zip(lengths, counts, slots, new):
        pages = [order.pop() for _ in range(count)]
        table[slot, :count] = torch.tensor(pages)
        flat = cache[pages].permute(1, 0, 3, 2, 4).reshape(2, count * page, hkv, d)[:, :length].double()
        keys.append(flat[0]), values.append(flat[1])
        queries.append(torch.randn(fresh, hq, d, generator=g).to(dtype))
        positions += range(length - fresh, length)
        token_slot += [slot] * fresh
    return {"q": torch.cat(queries).reshape(-1, hq * d).to(DEVICE), "cache": cache.to(DEVICE), "table": table.to(DEVICE), "keys": keys, "values": values,
            "queries": queries, "slots": torch.tensor(slots, dtype=torch.int32, device=DEVICE),
            "positions": torch.tensor(positions, dtype=torch.int32, device=DEVICE), "token_slot": torch.tensor(token_slot, dtype=torch.int32, device=DEVICE)}


def _plain_attention(case, hq, hkv, lengths, new, scale, chunk, sink, gate):
    rows, at = [], 0
    for key, value, query, length, fresh in zip(case["keys"], case["values"], case["queries"], lengths, new):
        for offset in range(fresh):
            i = length - fresh + offset
            first = i // chunk * chunk if chunk else 0
            k, v = (t[first : i + 1].repeat_interleave(hq // hkv, dim=1) for t in (key, value))
            scores = torch.einsum("hd,jhd->hj", query[offset].double(), k) * scale
            scores = torch.cat([scores, sink.double().cpu()[:, None]], dim=1) if sink is not None else scores
            weights = torch.softmax(scores, dim=1)[:, : k.shape[0]]
            row = torch.einsum("hj,jhd->hd", weights, v)
            if gate is not None:
                row = row * torch.sigmoid(gate[at].double().cpu())[:, None]
            rows.append(row.reshape(-1))
            at += 1
    return torch.stack(rows).float()


def _dressed(case, hq, d, dtype, seed, gated=True):
    """Sink, gate and an output that are what the engine hands over: the gate and the output columns of wider rows."""
    g = torch.Generator().manual_seed(seed)
    tokens = case["q"].shape[0]
    wide = torch.full((tokens, hq * d + 40), 7.0, dtype=dtype, device=DEVICE)
    gates = torch.randn(tokens, hq + 5, generator=g).to(dtype).to(DEVICE)
    return (torch.randn(hq, generator=g) * 2).to(DEVICE), gates[:, 2 : 2 + hq] if gated else None, wide


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hq,hkv,d,page,chunk", [(4, 2, 16, 16, 24), (6, 1, 32, 8, 1), (8, 2, 128, 16, 100), (6, 3, 64, 4, 0), (3, 3, 272, 16, 7)])
def test_one_warp_per_row_attention_in_chunks_with_sink_and_gate(hq, hkv, d, page, chunk, dtype):
    from rapid_llm_b200.ops import kernels

    lengths, new = [1, 15, 24, 25, 129, 200], [1, 15, 1, 2, 129, 33]
    case = _case(dtype, hq, hkv, d, page, lengths, new, seed=d + page)
    sink, gate, wide = _dressed(case, hq, d, dtype, seed=d)
    out, fault = wide[:, 8 : 8 + hq * d], _word()
    kernels.attention_generic(case["q"], case["cache"], out, positions=case["positions"], token_slot=case["token_slot"], block_table=case["table"],
                              num_heads=hq, num_kv_heads=hkv, head_dim=d, window=0, chunk=chunk, scale=d ** -0.5, fault=fault, sink=sink, gate=gate)
    assert int(fault.item()) == 0
    want = _plain_attention(case, hq, hkv, lengths, new, d ** -0.5, chunk, sink, gate)
    bound = {"rtol": 1e-4, "atol": 2e-5} if dtype == torch.float32 else {"rtol": 3e-2, "atol": 8e-3}
    torch.testing.assert_close(out.float().cpu(), want, **bound)
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + hq * d :] == 7).all(), "columns beside the output were written"


def _tiles(case, hq, hkv, d, page, lengths, new, chunk, sink, gate, out, splits=None, decode_kernel="auto"):
    from rapid_llm_b200.ops import kernels
    from rapid_llm_b200.parts.attention import AttentionItems
    from rapid_llm_b200.parts.base import StepShape

    starts = np.asarray(lengths, np.int32) - np.asarray(new, np.int32)
    plan = AttentionItems(hq // hkv, hkv, d, chunk=chunk).plan(StepShape(np.asarray(new, np.int32), starts, decode_only=max(new) == 1, page_size=page))
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
        window=0, chunk=chunk, scale=d ** -0.5, fault=fault, decode_kernel=decode_kernel, decode_rows=plan["decode_rows"], chunk_rows=plan["chunk_rows"],
        decode_splits=plan["decode_splits"], sink=sink, gate=gate)
    assert int(fault.item()) == 0
    return plan


@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("hq,hkv,d,page,chunk,splits", [
    (8, 2, 128, 16, 100, None), (8, 2, 128, 16, 300, None), (12, 3, 128, 8, 77, None), (8, 2, 128, 16, 0, None), (4, 4, 128, 64, 1, None),
    (6, 1, 32, 8, 40, None), (6, 1, 32, 8, 40, 3), (7, 7, 48, 4, 129, 2), (4, 2, 64, 16, 64, None), (3, 1, 256, 64, 90, None), (40, 2, 64, 16, 150, 4)])
def test_prompt_and_decode_tiles_in_chunks_with_sink_and_gate(hq, hkv, d, page, chunk, splits, gated):
    """Portions of prompts beside single tokens: the tcgen05 tiles at heads of 128 (unsplit portions, single tokens with
    key ranges of their own), the mma.sync tiles elsewhere, whole and with split key ranges; tiles that hold the border
    of two chunks, rows that see one key, a key range that begins inside a block."""
    lengths, new = [1, 15, 16, 17, 129, 200, 64, 700, 333, 301], [1, 15, 1, 2, 129, 1, 33, 1, 170, 1]
    case = _case(torch.bfloat16, hq, hkv, d, page, lengths, new, seed=d + page)
    sink, gate, wide = _dressed(case, hq, d, torch.bfloat16, seed=d, gated=gated)
    out = wide[:, 8 : 8 + hq * d]
    plan = _tiles(case, hq, hkv, d, page, lengths, new, chunk, sink, gate, out, splits)
    assert plan["chunk_rows"] == (256 if d == 128 else 64)
    want = _plain_attention(case, hq, hkv, lengths, new, d ** -0.5, chunk, sink, gate)
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=8e-3)
    assert (wide[:, :8] == 7).all() and (wide[:, 8 + hq * d :] == 7).all(), "columns beside the output were written"


@pytest.mark.parametrize("decode_kernel", ["auto", "mma", "deep", "shallow"])
@pytest.mark.parametrize("hq,hkv,page,chunk,splits,lengths", [
    (32, 8, 16, 512, None, [1, 5, 128, 513, 1000, 257, 2049]), (8, 2, 16, 700, 3, [700, 701, 1]), (40, 2, 64, 0, 2, [400, 90]),
    (8, 1, 16, 3000, 10, [5000]), (8, 2, 16, 2999, 16, [2998, 40]), (16, 4, 128, 1, None, [900, 3]), (4, 4, 8, 130, 1, [131, 260, 130])])
def test_single_tokens_on_the_decode_tiles_in_chunks_with_sink_and_gate(hq, hkv, page, chunk, splits, lengths, decode_kernel):
    """A sink counts once however many key ranges a row has and however they are merged: inside a CTA, inside a cluster
    (of up to sixteen CTAs, some without a key), by the merge kernel."""
    d, new = 128, [1] * len(lengths)
    case = _case(torch.bfloat16, hq, hkv, d, page, lengths, new, seed=page + hq)
    sink, gate, wide = _dressed(case, hq, d, torch.bfloat16, seed=hq)
    out = wide[:, : hq * d]
    _tiles(case, hq, hkv, d, page, lengths, new, chunk, sink, gate, out, splits, decode_kernel)
    want = _plain_attention(case, hq, hkv, lengths, new, d ** -0.5, chunk, sink, gate)
    torch.testing.assert_close(out.float().cpu(), want, rtol=3e-2, atol=8e-3)


def test_a_window_and_chunks_together_are_refused():
    from rapid_llm_b200.ops import kernels

    case = _case(torch.bfloat16, 2, 1, 32, 8, [20], [20], seed=1)
    out = torch.empty_like(case["q"])
    with pytest.raises(kernels.KernelError, match="invalid value"):
        kernels.attention_generic(case["q"], case["cache"], out, positions=case["positions"], token_slot=case["token_slot"], block_table=case["table"],
                                  num_heads=2, num_kv_heads=1, head_dim=32, window=4, chunk=4, scale=0.2, fault=_word())
