"""The Mozetar design's mechanisms one by one on the GPU, each kernel against the plain restatement (``plain_mozetar.py``)."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import plain_mozetar as plain

pytestmark = pytest.mark.gpu


def on(tensor: torch.Tensor, dtype: torch.dtype = torch.float32) -> torch.Tensor:
    return tensor.to(device="cuda", dtype=dtype).contiguous()


def ints(values) -> torch.Tensor:
    return torch.tensor(list(values), dtype=torch.int32, device="cuda")


def zero_status() -> torch.Tensor:
    return torch.zeros(1, dtype=torch.int32, device="cuda")


def close(got: torch.Tensor, want: torch.Tensor, limit: float, what=None) -> None:
    got, want = got.double().cpu(), want.double().cpu()
    assert bool(torch.isfinite(got).all()), what
    error = float((got - want).abs().max() / want.abs().max())
    assert error < limit, (what, error)


LIMIT = {torch.float32: 2e-5, torch.bfloat16: 1.5e-2}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8])
def test_streams_written_read_and_normed(streams, dtype):
    """One step between two sublayers: from equal streams and from unequal ones, the output as a tensor, with a bias, as a product's K slices,
    as routed experts' outputs, or nothing to write; widths with and without a 16-byte stride; chosen rows."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(streams)
    for tokens, dim in ((5, 72), (70, 130), (3, 33), (2, 2052)):
        mix, write, read = torch.randn(streams, streams, generator=generator), torch.randn(streams, generator=generator), torch.randn(streams, generator=generator)
        weight, bias = 1.0 + 0.2 * torch.randn(dim, generator=generator), torch.randn(dim, generator=generator)
        y = torch.randn(tokens, dim, generator=generator).to(dtype)
        experts, top = 4, 3
        pair_out, pair_weight = torch.randn(tokens * top, dim, generator=generator), torch.rand(tokens, top, generator=generator)
        chosen = torch.randint(0, experts, (tokens, top), generator=generator).to(torch.int32)
        partials = torch.randn(6, tokens, dim, generator=generator)
        forms = {
            "tensor": (on(y, dtype), y.double()),
            "bias": (ops.BiasedSum(on(y, dtype), on(bias)), y.double() + bias.double()),
            "experts": (ops.ExpertSum(on(pair_out), on(pair_weight), chosen.cuda(), experts, dtype), (pair_out.double().reshape(tokens, top, dim) * pair_weight.double()[:, :, None]).sum(1)),
        }
        if dtype == torch.bfloat16:
            total = partials.sum(0).to(dtype).double()
            forms["slices"] = (ops.SlicedSum(on(partials), dtype), total)
            forms["slices and bias"] = (ops.BiasedSum(ops.SlicedSum(on(partials), dtype), on(bias)), total + bias.double())
        for equal in (True, False):
            start = torch.randn(tokens, dim, generator=generator) if equal else torch.randn(tokens, streams, dim, generator=generator)
            X = start.double()[:, None, :].expand(-1, streams, -1) if equal else start.double()
            normed = lambda X: plain.rms_norm(plain.read_streams(X, read.double()), weight.double(), 1e-5)
            state = ops.ResidualStreams(on(start), streams)
            h = ops.stream_step(state, None, on(read), on(weight), 1e-5, dtype)
            close(h, normed(X), LIMIT[dtype])
            assert state.equal == equal
            for name, (output, value) in forms.items():
                state = ops.ResidualStreams(on(start), streams)
                update = ops.StreamWrite(output, on(mix), on(write))
                fresh = plain.write_streams(X, mix.double(), write.double(), value)
                rows = [tokens - 1, 0, tokens // 2]
                h = ops.stream_step(state, update, on(read), on(weight), 1e-5, dtype, keep=False, rows=ints(rows + [0]), num_rows=3)
                close(h, normed(fresh)[rows], LIMIT[dtype], name)
                assert torch.equal(state.tensor.cpu(), start)   # only looked at
                h = ops.stream_step(state, update, on(read), on(weight), 1e-5, dtype)
                close(h, normed(fresh), LIMIT[dtype], name)
                close(state.tensor, fresh, 1e-2 if name.startswith("slices") else 2e-6, name)   # (a slice sum may round the other way)
                assert not state.equal


def convolution_case(dtype, taps, channels, lengths, stride, add_input, generator):
    """Portions of these lengths behind states that are not zero; rows wider than the channels; returns what the kernel made and what is right."""
    from lalamo_b200 import ops

    tokens, slots = sum(lengths), [4, 0, 6, 2, 5][: len(lengths)]
    x = torch.randn(tokens, stride, generator=generator).to(dtype)
    weight = torch.randn(channels, taps, generator=generator)
    state = torch.randn(7, max(taps - 1, 1), channels, generator=generator).to(dtype)
    starts = np.cumsum([0] + lengths[:-1]).tolist()
    device_state = on(state, dtype) if taps > 1 else None
    status = zero_status()
    got = ops.causal_conv(on(x, dtype), device_state, on(weight), channels=channels, add_input=add_input, segment_start=ints(starts), segment_length=ints(lengths),
                          segment_slot=ints(slots), segments=len(lengths), max_length=max(lengths), status=status)
    assert int(status.item()) == 0
    want_state = state.clone()
    pieces = []
    for start, length, slot in zip(starts, lengths, slots):
        rows = x[start : start + length, :channels].double()
        history = state[slot].double() if taps > 1 else rows[:0]
        joined = torch.cat([history, rows])
        y = plain.causal_conv(joined, weight.double())[history.shape[0] :]
        pieces.append(y + rows if add_input else y)
        if taps > 1:
            want_state[slot] = joined[-(taps - 1) :].to(dtype)
    close(got, torch.cat(pieces), LIMIT[dtype], (taps, channels, lengths))
    if taps > 1:
        assert torch.equal(device_state.cpu(), want_state), (taps, channels, lengths)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_causal_convolution_over_portions(dtype):
    """All numbers of taps, channels of 16-byte multiples and others, portions shorter than the taps, just as long, and over several blocks."""
    generator = torch.Generator().manual_seed(2)
    for taps in (1, 2, 3, 4, 5, 9, 17):
        for channels, stride in ((64, 64), (24, 40), (13, 13), (1032, 1032)):
            for lengths in ([1], [1, 2, 3, 1, 40], [taps, 16, 17, max(1, taps - 1)], [33, 1]):
                convolution_case(dtype, taps, channels, lengths, stride, add_input=taps % 2 == 0, generator=generator)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_input_convolution_inside_the_stream_step(dtype):
    """For single tokens the convolution runs where the norm is computed: the same values and the same states as the kernel of its own."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(3)
    for taps in (1, 2, 4, 6):
        for dim in (64, 33):
            tokens, slots = 4, [3, 0, 5, 1]
            x = torch.randn(tokens, 2, dim, generator=generator)
            weight, conv_weight, read = 1.0 + 0.2 * torch.randn(dim, generator=generator), torch.randn(dim, taps, generator=generator), torch.randn(2, generator=generator)
            state = torch.randn(6, taps - 1, dim, generator=generator).to(dtype) if taps > 1 else None
            mine, theirs = (on(state, dtype), on(state, dtype)) if taps > 1 else (None, None)
            status = zero_status()
            conv = dict(weight=on(conv_weight), state=mine, token_segment=ints(range(tokens)), segment_slot=ints(slots), status=status)
            fused = ops.stream_step(ops.ResidualStreams(on(x), 2), None, on(read), on(weight), 1e-5, dtype, conv=conv)
            h = ops.stream_step(ops.ResidualStreams(on(x), 2), None, on(read), on(weight), 1e-5, dtype)
            apart = ops.causal_conv(h, theirs, on(conv_weight), add_input=True, segment_start=ints(range(tokens)), segment_length=ints([1] * tokens),
                                    segment_slot=ints(slots), segments=tokens, max_length=1, status=status)
            close(fused, apart, 1e-6 if dtype == torch.float32 else 8e-3)
            assert int(status.item()) == 0 and (taps == 1 or torch.equal(mine, theirs))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_polynomial_of_norms(dtype):
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(4)
    coefficients = torch.tensor([0.7, -0.4, 0.9, 0.2])
    for rows, dim in ((1, 8), (3, 75), (70, 264), (2, 9000), (600, 72)):
        z = (2.0 * torch.randn(rows, dim, generator=generator)).to(dtype)
        z[0] *= 1e-3   # eps matters
        close(ops.poly_norm(on(z, dtype), on(coefficients), 1e-5), plain.poly_norm(z.double(), coefficients.double(), 1e-5), LIMIT[dtype], (rows, dim))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_combining_two_maps(dtype):
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(5)
    for tokens, heads, groups, vd in ((3, 4, 2, 16), (70, 6, 1, 24), (2, 3, 3, 10), (9, 8, 2, 128), (1, 2, 1, 520)):
        maps = torch.randn(tokens, groups, 2, heads // groups, vd, generator=generator)
        wide = torch.randn(tokens, heads + 11, generator=generator).to(dtype)
        out = torch.empty(tokens, heads * vd, dtype=dtype, device="cuda")
        ops.combine_maps(on(maps), on(wide, dtype)[:, 5 : 5 + heads], out, num_heads=heads, num_groups=groups, value_dim=vd, lam=0.8, eps=1e-5, factor=0.6)
        a = maps.double().transpose(1, 2).reshape(tokens, 2, heads, vd)
        want = plain.combine_maps(a[:, 0], a[:, 1], 0.8, 0.4, wide.double()[:, 5 : 5 + heads], 1e-5)
        close(out, want.reshape(tokens, -1), LIMIT[dtype], (tokens, heads, groups, vd))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_forget_recurrence(dtype):
    """Portions of unequal lengths from states that are not zero (one long enough for chunks side by side), head sizes of all kinds,
    gates that hardly forget: what they write keeps its precision."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(6)
    for heads, dk, dv, lengths in ((3, 12, 20, [5, 1, 37]), (2, 40, 8, [2, 3, 9]), (1, 64, 64, [60, 1, 1]), (2, 16, 32, [900, 1, 3])):
        tokens, start_f = sum(lengths), -(-(heads * (dk + dv)) // 8) * 8
        proj = torch.randn(tokens, start_f + heads * dk, generator=generator).to(dtype)
        bias, lower = 4.0 + 3.0 * torch.randn(heads * dk, generator=generator), torch.rand(heads * dk, generator=generator)
        weight, state = 1.0 + 0.1 * torch.randn(dv, generator=generator), torch.randn(5, heads, dk, dv, generator=generator)
        slots, starts = [3, 0, 4], np.cumsum([0] + lengths[:-1]).tolist()
        device_state, device_proj, status = on(state), on(proj, dtype), zero_status()
        host = ops.gated_delta_chunk_plan(starts, lengths)
        plan = {name: ints(array.tolist()) for name, array in host.items()}
        plan.update(num_chunks=host["chunk_start"].size, num_long=host["long_table"].size // 3, num_direct=host["direct"].size)
        out = ops.linear_attention(device_proj, device_state, num_heads=heads, key_dim=dk, value_dim=dv, decay_logits=device_proj[:, start_f:], decay_bias=on(bias),
                                   lower=on(lower), query_silu=True, norm_weight=on(weight), norm_eps=1e-5, gate_offset=None, segment_start=ints(starts),
                                   segment_length=ints(lengths), segment_slot=ints(slots), segments=3, status=status, chunk_plan=plan)
        assert int(status.item()) == 0
        for start, length, slot in zip(starts, lengths, slots):
            rows = proj[start : start + length].double()
            q = plain.silu(rows[:, : heads * dk]).reshape(length, heads, dk)
            v = rows[:, heads * dk : heads * (dk + dv)].reshape(length, heads, dv)
            f = plain.forget_gate(rows[:, start_f:] + bias.double(), lower.double()).reshape(length, heads, dk)
            want, last = plain.forget_recurrence(q, f, v, state[slot].double())
            close(out[start : start + length], plain.rms_norm(want, weight.double(), 1e-5).reshape(length, -1), 10 * LIMIT[dtype] if dtype == torch.float32 else LIMIT[dtype])
            close(device_state[slot], last, 1e-5)


def test_router_with_groups_scored_by_their_largest():
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(7)
    differs = 0
    for experts, top, count, keep in ((6, 2, 3, 1), (12, 3, 4, 2), (8, 2, 2, 1), (5, 3, 1, 1), (4, 1, 4, 2)):
        for tokens in (40, 600):
            x, router = torch.randn(tokens, 72, generator=generator), torch.randn(experts, 72, generator=generator) / 4
            chosen, weights = ops.moe_route(on(x), on(router), top=top, group_count=count, group_keep=keep, score="softmax", renormalize=True, group_score="largest")
            scores = torch.softmax(x.double() @ router.double().T, dim=-1)
            want = torch.tensor([plain.choose_experts(scores[t], {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}) for t in range(tokens)])
            assert torch.equal(chosen.cpu().long(), want), (experts, top, count, keep)
            picked = torch.gather(scores, 1, want)
            assert torch.allclose(weights.cpu().double(), picked / picked.sum(1, keepdim=True), rtol=1e-5)
            other, _ = ops.moe_route(on(x), on(router), top=top, group_count=count, group_keep=keep, score="softmax", renormalize=True)
            differs += int((other != chosen).any())
    assert differs >= 4   # the sum of a group's two largest would have chosen others


def attention_case(dtype, heads, groups, kd, vd, value_groups, window, contexts, lengths, kernel, out_dtype, seed, page_size=16):
    """One step's attention over requests that hold ``contexts`` tokens and bring ``lengths`` more, against the plain attention; scattered pages, and
    every row that nobody may read (past a request's last position, before a window, foreign pages) is NaN.  One key per request, far
    from most queries, stands out in its score."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(seed)
    totals = [c + n for c, n in zip(contexts, lengths)]
    blocks = -(-max(totals) // page_size)
    pages = blocks * len(totals) + 2
    order = torch.randperm(pages, generator=generator).tolist()
    table = [[order[r * blocks + b] for b in range(blocks)] for r in range(len(totals))]
    k_pages = torch.full((pages, page_size, groups, kd), float("nan"), dtype=dtype)
    v_pages = torch.full((pages, value_groups, vd, page_size), float("nan"), dtype=dtype)
    queries, wants = [], []
    for r, (context, length, total) in enumerate(zip(contexts, lengths, totals)):
        k = torch.randn(total, groups, kd, generator=generator).to(dtype)
        v = torch.randn(total, value_groups, vd, generator=generator).to(dtype)
        q = torch.randn(length, heads, kd, generator=generator).to(dtype)
        mark = int(torch.randint(0, total, (1,), generator=generator))
        k[mark] = (4.0 * k[mark].float()).to(dtype)
        oldest = 0 if window is None else max(0, context - window + 1)
        for position in range(oldest, total):
            page, row = table[r][position // page_size], position % page_size
            k_pages[page, row], v_pages[page, :, :, row] = k[position], v[position]
        each = groups // value_groups
        want = torch.zeros(length, heads, vd, dtype=torch.float64)
        i, j = torch.arange(context, total)[:, None], torch.arange(total)[None]
        seen = (j <= i) if window is None else (j <= i) & (i - j < window)
        for head in range(heads):
            g = head // (heads // groups)
            score = q[:, head].double() @ k[:, g].double().T * kd**-0.5
            want[:, head] = torch.softmax(score.masked_fill(~seen, float("-inf")), dim=1) @ v[:, g // each].double()
        queries.append(q.reshape(length, heads * kd))
        wants.append(want.reshape(length, heads * vd))
    tokens = sum(lengths)
    q = on(torch.cat(queries), dtype)
    out = torch.full((tokens, heads * vd), float("nan"), dtype=out_dtype, device="cuda")
    status = zero_status()
    common = dict(positions=ints(p for c, n in zip(contexts, lengths) for p in range(c, c + n)), token_segment=ints(r for r, n in enumerate(lengths) for _ in range(n)),
                  block_table=torch.tensor(table, dtype=torch.int32, device="cuda"), num_heads=heads, num_groups=groups, head_dim=kd, scale=kd**-0.5, window=window,
                  status=status, value_dim=vd, value_groups=value_groups)
    k_pages, v_pages = on(k_pages, dtype), on(v_pages, dtype)
    if kernel == "plain":
        ops.paged_attention_plain(q, k_pages, v_pages, out, **common)
    elif kernel == "alone":
        ops.attention_decode(q, k_pages, v_pages, out, max_context=max(totals), **common)
    elif kernel == "two maps":   # two consecutive key heads are one row of the cache
        ops.attention_decode(q, k_pages.view(pages, page_size, value_groups, 2 * kd), v_pages, out, max_context=max(totals),
                             **dict(common, num_groups=value_groups, head_dim=2 * kd, two_maps=True))
    else:
        starts = np.cumsum([0] + lengths[:-1]).tolist()
        tiles = [value for start, n in zip(starts, lengths) for first in range(start, start + n, 32) for value in (first, min(32, start + n - first))]
        ops.attention_prefill(q, k_pages, v_pages, out, tiles=ints(tiles), num_tiles=len(tiles) // 2, kernel=None if kernel == "tiles" else kernel, **common)
    assert int(status.item()) == 0
    close(out, torch.cat(wants), 3e-5 if dtype == torch.float32 else 1.2e-2 if out_dtype == torch.bfloat16 else 8e-3, (heads, groups, kd, vd, value_groups, window, kernel))


SHAPES = [   # query heads, key heads, channels of a key and of a value head, value heads
    (8, 4, 16, 24, 2), (6, 2, 16, 40, 1), (4, 4, 64, 128, 2), (8, 2, 32, 64, 1), (16, 2, 64, 64, 1), (4, 1, 96, 40, 1), (12, 6, 48, 96, 3), (8, 2, 128, 72, 2),
    (6, 2, 80, 16, 2), (24, 2, 48, 128, 1), (2, 2, 40, 64, 1), (48, 2, 16, 8, 1), (4, 2, 64, 64, 2),
]
STEPS = [([0, 0, 15, 16, 31], [1, 2, 1, 1, 1]), ([0, 5, 63, 64], [70, 33, 40, 17]), ([200, 64, 39, 40, 0], [1, 17, 1, 1, 90])]


@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("window", [None, 1, 20, 40, 65])
def test_attention_over_keys_and_values_of_different_sizes(shape, window):
    """Every kernel that takes the shape: the plain one in both types, tokens that attend alone, both maps of a row at once, tiles."""
    from lalamo_b200 import ops

    heads, groups, kd, vd, value_groups = shape
    for index, (contexts, lengths) in enumerate(STEPS):
        case = dict(heads=heads, groups=groups, kd=kd, vd=vd, value_groups=value_groups, window=window, contexts=contexts, lengths=lengths, seed=10 * index + heads)
        attention_case(torch.float32, kernel="plain", out_dtype=torch.float32, **case)
        attention_case(torch.bfloat16, kernel="plain", out_dtype=torch.float32, **case)
        if ops.decode_attention_supported(torch.bfloat16, kd, 16, vd):
            for out_dtype in (torch.bfloat16, torch.float32):
                attention_case(torch.bfloat16, kernel="alone", out_dtype=out_dtype, **case)
        if groups == 2 * value_groups and ops.decode_attention_supported(torch.bfloat16, 2 * kd, 16, vd):
            attention_case(torch.bfloat16, kernel="two maps", out_dtype=torch.float32, **case)
        if ops.wide_prefill_attention_supported(torch.bfloat16, heads, groups, kd, vd, 16):
            attention_case(torch.bfloat16, kernel="tiles", out_dtype=torch.float32, **case)
            attention_case(torch.bfloat16, kernel="tiles", out_dtype=torch.bfloat16, **case)
        if ops.prefill_attention_supported(torch.bfloat16, heads, groups, kd, 16):
            attention_case(torch.bfloat16, kernel="mma", out_dtype=torch.float32, **case)


def test_attention_over_larger_pages_and_many_keys():
    for kernel, (heads, groups, kd, vd, value_groups) in (("tiles", (4, 4, 64, 128, 2)), ("two maps", (4, 4, 64, 128, 2)), ("mma", (4, 1, 96, 40, 1)), ("alone", (4, 1, 96, 40, 1))):
        attention_case(torch.bfloat16, heads, groups, kd, vd, value_groups, None, [1500, 0], [20, 3], kernel, torch.float32, 3, page_size=48)
        attention_case(torch.bfloat16, heads, groups, kd, vd, value_groups, 300, [700, 1200], [40, 33], kernel, torch.float32, 4, page_size=32)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens", [3, 70, 530])
def test_rewriting_heads_with_a_temperature_and_shared_values(dtype, tokens):
    """Queries, keys and values laid out from a projection's rows: few tokens, many, and runs of tokens; rotated and not; sizes of 16-byte
    multiples and others; queries alone; positions that begin inside a page and a request's border inside a run."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(tokens)
    page_size = 16
    for heads, groups, kd, vd, value_groups, rotary, every in ((4, 4, 16, 24, 2, 0, 5), (3, 1, 48, 16, 1, 32, 0), (2, 2, 12, 10, 2, 4, 7), (8, 2, 64, 128, 1, 64, 64), (2, 2, 24, 24, 1, 8, 3)):
        first = tokens // 3
        lengths, contexts = [first, tokens - first], [5, 2]
        columns = heads * kd + groups * kd + value_groups * vd
        wide = torch.randn(tokens, columns + 8, generator=generator).to(dtype)
        positions = [p for c, n in zip(contexts, lengths) for p in range(c, c + n)]
        segments = [r for r, n in enumerate(lengths) for _ in range(n)]
        blocks = -(-(max(c + n for c, n in zip(contexts, lengths))) // page_size)
        table = torch.randperm(2 * blocks, generator=generator).reshape(2, blocks).to(torch.int32)
        freq = plain.frequencies({"dims": rotary, "base": 100.0}).float() if rotary else None

        def turned(x):   # halves: channel i with i + rotary / 2
            if not rotary:
                return x
            angle = torch.tensor(positions, dtype=torch.float64)[:, None] * freq.double()[None]
            cos, sin, u, v = torch.cos(angle)[:, None], torch.sin(angle)[:, None], x[..., : rotary // 2], x[..., rotary // 2 : rotary]
            return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., rotary:]], dim=-1)

        rows = wide.double()
        factor = plain.query_temperature(torch.tensor(positions), {"coef": 0.6, "every": every} if every else None)
        want_q = turned(rows[:, : heads * kd].reshape(tokens, heads, kd)) * factor[:, None, None]
        want_k = turned(rows[:, heads * kd : (heads + groups) * kd].reshape(tokens, groups, kd))
        want_v = rows[:, (heads + groups) * kd : columns].reshape(tokens, value_groups, vd)
        for write in (True, False):
            q = torch.full((tokens, heads * kd), float("nan"), dtype=dtype, device="cuda")
            k_pages = torch.full((2 * blocks, page_size, groups, kd), 7.0, dtype=dtype, device="cuda")
            v_pages = torch.full((2 * blocks, value_groups, vd, page_size), 7.0, dtype=dtype, device="cuda")
            status = zero_status()
            ops.qk_norm_rope_write(on(wide, dtype)[:, :columns] if write else on(wide[:, : heads * kd], dtype), q, k_pages, v_pages, q_weight=None, k_weight=None, eps=0.0,
                                   scale_offset=0.0, inv_freq=on(freq) if rotary else None, rotary_dim=rotary, positions=ints(positions), token_segment=ints(segments),
                                   block_table=table.cuda(), num_heads=heads, num_groups=groups, head_dim=kd, write_kv=write, status=status, value_dim=vd,
                                   value_groups=value_groups, temperature=0.6, temperature_every=every)
            assert int(status.item()) == 0
            close(q, want_q.reshape(tokens, -1), 3e-5 if dtype == torch.float32 else 8e-3, (heads, groups, kd, vd))
            if not write:
                assert bool((k_pages == 7.0).all()) and bool((v_pages == 7.0).all())
                continue
            place = [(int(table[s, p // page_size]), p % page_size) for s, p in zip(segments, positions)]
            page, row = torch.tensor([x for x, _ in place]), torch.tensor([x for _, x in place])
            close(k_pages.cpu()[page, row], want_k, 3e-5 if dtype == torch.float32 else 8e-3)
            assert torch.equal(v_pages.cpu()[page, :, :, row].double(), want_v)
            touched = torch.zeros(2 * blocks, page_size, dtype=torch.bool)
            touched[page, row] = True
            assert bool((k_pages.cpu()[~touched] == 7.0).all()) and bool((v_pages.cpu().permute(0, 3, 1, 2)[~touched] == 7.0).all())
