"""The Zevetar design's mechanisms one by one on the GPU, each kernel against the plain restatement (``plain_zevetar.py``)."""

from __future__ import annotations

import numpy as np
import pytest
import torch

import plain_zevetar as plain

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
@pytest.mark.parametrize("tokens,dim", [(1, 64), (5, 70), (70, 130), (3, 33), (2, 4100), (200, 1024)])
def test_terms_added_to_the_stream_and_normed(tokens, dim, dtype):
    """One to three terms as tensors, a product's K slices or routed experts' outputs, with and without a vector and a number per token; the
    norm of the sum or only the sum; chosen rows, which leave the stream as it is.  Experts that do not exist leave unwritten memory unread."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(tokens + dim)
    normal = lambda *shape: torch.randn(*shape, generator=generator)
    experts, top = 4, 6
    y, z = normal(tokens, dim).to(dtype), normal(tokens, dim).to(dtype)
    pair_out, pair_weight = normal(tokens * top, dim), torch.rand(tokens, top, generator=generator)
    chosen = torch.randint(0, experts, (tokens, top), generator=generator).to(torch.int32)
    chosen[0, 2] = experts   # no expert: its row is never read
    pair_out[2] = float("nan")
    kept = pair_out.double().reshape(tokens, top, dim).clone()
    kept[0, 2] = 0.0
    partials = normal(6, tokens, dim)
    scale, other_scale, gate = normal(dim), normal(dim), torch.rand(tokens, 1, generator=generator)
    values = {
        "tensor": (on(y, dtype), y.double()),
        "experts": (ops.ExpertSum(on(pair_out), None, chosen.cuda(), experts, dtype), kept.sum(1)),
        "weighed experts": (ops.ExpertSum(on(pair_out), on(pair_weight), chosen.cuda(), experts, dtype), (kept * pair_weight.double()[:, :, None]).sum(1)),
    }
    if dtype == torch.bfloat16:
        values["slices"] = (ops.SlicedSum(on(partials), dtype), partials.sum(0).to(dtype).double())
    weight, start = 1.0 + 0.2 * normal(dim), normal(tokens, dim)
    second = (on(z, dtype), z.double())
    for name, first in values.items():
        for terms in (
            [(first, None, None)],
            [(first, scale, None)],
            [(second, scale, None), (first, other_scale, gate)],
            [(first, scale, gate), (second, None, None), (first, other_scale, None)],
        ):
            total = start.double()
            for (_, value), vector, number in terms:
                total = total + (1.0 if vector is None else vector.double()) * ((1.0 if number is None else number.double()) * value)
            given = ops.TermSum([ops.ResidualTerm(made, None if vector is None else on(vector), None if number is None else on(number)) for (made, _), vector, number in terms])
            limit = 1e-2 if name == "slices" else 2e-6   # (a slice sum may round the other way)
            stream = on(start)
            rows = [tokens - 1, 0, tokens // 2]
            out = torch.empty(3, dim, dtype=dtype, device="cuda")
            ops.residual_terms(stream, given, on(weight), 1e-5, out, rows=ints(rows + [0]), num_rows=3, write_back=False)
            close(out, plain.rms_norm(total[rows], weight.double(), 1e-5), LIMIT[dtype], name)
            assert torch.equal(stream.cpu(), start)   # only looked at
            out = torch.empty(tokens, dim, dtype=dtype, device="cuda")
            ops.residual_terms(stream, given, on(weight), 1e-5, out)
            close(out, plain.rms_norm(total, weight.double(), 1e-5), LIMIT[dtype], name)
            close(stream, total, limit, name)
            alone = on(start)
            ops.residual_add(alone, given)
            assert torch.equal(alone, stream)
            close(given.sum(), total - start.double(), max(limit, 2e-6 if dtype == torch.float32 else 8e-3), name)


def test_terms_that_do_not_fit_are_refused():
    from lalamo_b200 import ops

    x = torch.zeros(4, 16, device="cuda")
    y = torch.zeros(4, 16, device="cuda")
    bad = [
        ops.TermSum([]),
        ops.TermSum([ops.ResidualTerm(y)] * 4),
        ops.TermSum([ops.ResidualTerm(torch.zeros(3, 16, device="cuda"))]),
        ops.TermSum([ops.ResidualTerm(y, scale=torch.zeros(8, device="cuda"))]),
        ops.TermSum([ops.ResidualTerm(y, gate=torch.zeros(3, device="cuda"))]),
        ops.TermSum([ops.ResidualTerm(y), ops.ResidualTerm(y.bfloat16())]),
    ]
    for terms in bad:
        with pytest.raises(ops.KernelError):
            ops.residual_terms(x, terms)
    with pytest.raises(ops.KernelError):
        ops.residual_terms(x, ops.TermSum([ops.ResidualTerm(y)]), torch.ones(16, device="cuda"), 1e-5, torch.zeros(2, 16, device="cuda"), rows=ints([0, 1]))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,latent,rope,heads,dim", [(24, 32, 8, 4, 16), (13, 27, 6, 3, 9), (200, 128, 32, 2, 64), (8, 272, 16, 1, 32)])
def test_query_latents_rows_and_rotated_queries(q_rank, latent, rope, heads, dim, dtype):
    """The norm of the query latent (zeros behind it), the row a token leaves, the queries' rotation, with a factor on sines and cosines; a
    layer that leaves no rows; positions far from zero, on both sides of a page's border."""
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(q_rank)
    rot = {"dims": rope, "base": 500.0, "scaling": {"factor": 6.0, "original": 300, "fast": 8.0, "slow": 1.0}}
    frequency, factor = plain.pair_frequencies(rot)
    positions = [0, 15, 16, 17, 900, 31]
    tokens, page_size = len(positions), 16
    stride = q_rank + latent + rope + 24
    product = torch.randn(tokens, stride, generator=generator).to(dtype)
    down_at = q_rank + 3
    q_weight, weight = 1.0 + 0.2 * torch.randn(q_rank, generator=generator), 1.0 + 0.2 * torch.randn(latent, generator=generator)
    segments = [0, 0, 1, 1, 0, 2]
    table = torch.full((3, 64), -1, dtype=torch.int32)
    for page, (segment, position) in enumerate(dict.fromkeys((s, p // page_size) for s, p in zip(segments, positions))):
        table[segment, position] = page + 1
    device = on(product, dtype)
    common = dict(inv_freq=on(frequency), turn_scale=factor, positions=ints(positions), token_segment=ints(segments), block_table=table.cuda())
    at = torch.tensor(positions)
    interleave = lambda x: torch.stack([x[..., : rope // 2], x[..., rope // 2 :]], dim=-1).reshape(x.shape)   # the kernels' order of channels into pairs of neighbours
    for writes in (True, False):
        pages = torch.full((8, page_size, 1, latent + rope), float("nan"), dtype=dtype, device="cuda")
        q_latent = torch.full((tokens, -(-q_rank // 32) * 32), float("nan"), dtype=dtype, device="cuda")
        status = zero_status()
        ops.latent_down(device[:, :q_rank], device[:, down_at : down_at + latent + rope] if writes else None, q_latent, pages, q_norm_weight=on(q_weight), q_eps=1e-5,
                        norm_weight=on(weight) if writes else None, eps=1e-4, scale_offset=0.0, latent=latent, rope=rope, status=status, **common)
        assert int(status.item()) == 0
        close(q_latent[:, :q_rank], plain.rms_norm(product[:, :q_rank].double(), q_weight.double(), 1e-5), LIMIT[dtype])
        assert float(q_latent[:, q_rank:].abs().sum()) == 0.0
        if not writes:
            assert bool(torch.isnan(pages).all())
            continue
        rows = torch.stack([pages[int(table[s, p // page_size]), p % page_size, 0] for s, p in zip(segments, positions)]).double().cpu()
        down = product[:, down_at : down_at + latent + rope].double()
        close(rows[:, :latent], plain.rms_norm(down[:, :latent], weight.double(), 1e-4), LIMIT[dtype])
        close(interleave(rows[:, latent:]), plain.rotate_neighbours(interleave(down[:, latent:]), at, rot), 1e-4 if dtype == torch.float32 else LIMIT[dtype])
        assert int(torch.isnan(pages).any(dim=-1).logical_not().sum()) == tokens   # nothing else was written
    q = torch.randn(tokens, heads * (dim + rope), generator=generator).to(dtype)
    q_in = torch.randn(heads, tokens, latent, generator=generator).to(dtype)
    queries = torch.empty(tokens, heads, latent + rope, dtype=dtype, device="cuda")
    ops.latent_prepare(on(q, dtype), on(q_in, dtype), None, queries, pages, norm_weight=None, eps=1e-5, scale_offset=0.0, num_heads=heads, head_dim=dim, latent=latent,
                       rope=rope, write_kv=False, status=status, **common)
    assert torch.equal(queries[..., :latent].cpu(), q_in.transpose(0, 1))
    turned = plain.rotate_neighbours(interleave(q.double().reshape(tokens, heads, dim + rope)[..., dim:]), at, rot)
    close(interleave(queries[..., latent:].double().cpu()), turned, 1e-4 if dtype == torch.float32 else LIMIT[dtype])


def retention_case(lengths, contexts, heads, dim, vdim, dims, dtype, generator, chunked=False):
    """Portions of these lengths at these positions behind states that are not zero; the read-outs and the states they leave."""
    from lalamo_b200 import ops

    tokens, slots = sum(lengths), [3, 0, 5, 1][: len(lengths)]
    rot = {"dims": dims, "base": 700.0}
    decay = [1.0 - 2.0 ** (-2 - head) for head in range(heads)]
    key_width, value_width = heads * dim, heads * vdim
    gate_offset = -(-(2 * key_width + value_width) // 8) * 8
    proj = torch.randn(tokens, gate_offset + value_width, generator=generator).to(dtype)
    state = torch.randn(6, heads, dim, vdim, generator=generator)
    starts = np.cumsum([0] + lengths[:-1]).tolist()
    positions = [context + i for length, context in zip(lengths, contexts) for i in range(length)]
    device_state, status = on(state), zero_status()
    plan = None
    if chunked:
        plan = ops.gated_delta_chunk_plan(starts, lengths, chunk_tokens=64, long_portion=100)
        plan = {**{name: torch.from_numpy(values).cuda() for name, values in plan.items()}, "num_chunks": plan["chunk_start"].size, "num_long": plan["long_table"].size // 3,
                "num_direct": plan["direct"].size, "chunk_tokens": 64}
    frequency, _ = plain.pair_frequencies(rot) if dims else (None, None)
    got = ops.linear_attention(on(proj, dtype), device_state, num_heads=heads, key_dim=dim, value_dim=vdim, fixed_decay=on(torch.tensor(decay)), key_scale=dim ** -0.5,
                               norm_weight=torch.ones(vdim, device="cuda"), norm_eps=1e-5, gate_offset=gate_offset, gate_activation="silu", segment_start=ints(starts),
                               segment_length=ints(lengths), segment_slot=ints(slots), segments=len(lengths), status=status, chunk_plan=plan,
                               inv_freq=on(frequency) if dims else None, positions=ints(positions))
    assert int(status.item()) == 0
    at = torch.tensor(positions)
    p = proj.double()
    q, k, v = p[:, :key_width].reshape(tokens, heads, dim), p[:, key_width : 2 * key_width].reshape(tokens, heads, dim), p[:, 2 * key_width : 2 * key_width + value_width].reshape(tokens, heads, vdim)
    if dims:
        q, k = plain.rotate_halves(q, at, rot), plain.rotate_halves(k, at, rot)
    k = k * dim ** -0.5
    out = torch.zeros(tokens, heads, vdim, dtype=torch.float64)
    wanted_state = state.double().clone()
    for start, length, slot in zip(starts, lengths, slots):
        S = wanted_state[slot]
        for t in range(start, start + length):
            S = torch.tensor(decay, dtype=torch.float64)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            out[t] = torch.einsum("hkv,hk->hv", S, q[t])
        wanted_state[slot] = S
    want = plain.rms(out, 1e-5).reshape(tokens, value_width) * plain.silu(p[:, gate_offset:])
    close(got, want, 3e-4 if dtype == torch.float32 else LIMIT[dtype], (lengths, dim, vdim, dims))
    close(device_state, wanted_state, 3e-5, (lengths, dim, vdim, dims))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,vdim,dims", [(4, 16, 24, 16), (2, 64, 128, 64), (3, 12, 20, 4), (1, 10, 6, 10), (2, 48, 32, 0), (2, 136, 40, 100)])
def test_rotated_retention_over_portions(heads, dim, vdim, dims, dtype):
    generator = torch.Generator().manual_seed(dim)
    for lengths, contexts in (([1], [0]), ([1, 1, 1], [7, 0, 500]), ([2, 33, 1], [3, 0, 64]), ([150, 17], [0, 31])):
        retention_case(lengths, contexts, heads, dim, vdim, dims, dtype, generator)
    retention_case([150, 17, 200], [40, 31, 0], heads, dim, vdim, dims, dtype, generator, chunked=True)


@pytest.mark.parametrize("path,dtype", [("plain", torch.float32), ("plain", torch.bfloat16), ("stream", torch.float32), ("stream", torch.bfloat16), ("grouped", torch.bfloat16)])
@pytest.mark.parametrize("tokens,width,ff,experts,top,gated", [(1, 72, 40, 6, 1, True), (5, 72, 40, 6, 3, True), (150, 128, 64, 6, 2, True), (37, 64, 104, 3, 3, False)])
def test_experts_weighed_on_their_input(tokens, width, ff, experts, top, gated, path, dtype):
    from lalamo_b200 import ops

    generator = torch.Generator().manual_seed(tokens)
    x = torch.randn(tokens, width, generator=generator).to(dtype)
    gate, up = (torch.randn(experts, ff, width, generator=generator).mul(2.0 / width ** 0.5).to(dtype) for _ in range(2))
    down = torch.randn(experts, width, ff, generator=generator).mul(ff ** -0.5).to(dtype)
    weights = 0.1 + torch.rand(tokens, top, generator=generator)
    chosen = torch.stack([torch.randperm(experts, generator=generator)[:top] for _ in range(tokens)]).to(torch.int32)
    want = torch.zeros(tokens, width, dtype=torch.float64)
    for t in range(tokens):
        for k in range(top):
            e, row = int(chosen[t, k]), float(weights[t, k]) * x[t].double()
            if gated:
                want[t] += plain.gated(row[None], {"gate": gate[e].double(), "up": up[e].double(), "down": down[e].double()})[0]
            else:
                want[t] += plain.silu(up[e].double() @ row) @ down[e].double().T
    arguments = (on(x, dtype), on(gate, dtype) if gated else None, on(up, dtype), on(down, dtype), chosen.cuda(), on(weights))
    close(ops.moe_experts(*arguments, "silu", path=path, weigh_input=True), want, 1e-5 if dtype == torch.float32 else 2e-2, path)
    routed = ops.moe_experts(*arguments, "silu", path=path, weigh_input=True, combine=False)
    assert routed.weights is None
    close(routed.sum(), want, 1e-5 if dtype == torch.float32 else 2e-2, path)
    stream = torch.ones(tokens, width, device="cuda")
    ops.moe_combine_add(routed, stream)
    close(stream, want + 1.0, 1e-5 if dtype == torch.float32 else 2e-2, path)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens", [1, 12, 130])
@pytest.mark.parametrize("width,ff,experts,top,shared_ff", [(64, 24, 6, 2, 32), (128, 64, 8, 1, 64), (70, 9, 5, 3, 11)])
def test_the_routed_feed_forward_as_a_sum_of_terms(width, ff, experts, top, shared_ff, tokens, dtype):
    """The part as a block runs it (terms left to the next norm), and as a plain output: router, choice, experts and gated shared expert."""
    from lalamo_b200 import ops
    from lalamo_b200.config import GatedMLPSpec, RoutedMLPSpec
    from lalamo_b200.parts.base import Runtime, build_part
    from lalamo_b200.parts.routed_mlp import RoutedMLP

    generator = torch.Generator().manual_seed(width)
    spec = RoutedMLPSpec(model_dim=width, hidden_dim=ff, num_experts=experts, top=top, weigh_input=True, shared=GatedMLPSpec(width, shared_ff), shared_gate=True)
    normal = lambda *shape: (torch.randn(*shape, generator=generator) / shape[-1] ** 0.5).to(torch.bfloat16)
    plain_names = {"router": "router", "shared_gate": "shared.sg", "shared.gate_proj": "shared.gate", "shared.up_proj": "shared.up", "shared.down_proj": "shared.down",
                   **{f"experts.{e}.{n}_proj": f"e{e}.{n}" for e in range(experts) for n in ("gate", "up", "down")}}
    tensors = {local: normal(*decl.shape) * (3.0 if local == "router" else 1.0) for local, decl in RoutedMLP.tensor_decls(spec).items()}
    part = build_part(spec, tensors, Runtime(torch.device("cuda"), dtype))
    x = torch.randn(tokens, width, generator=generator).to(dtype)
    chosen = ops.moe_route(on(x, dtype), part.router, top=top, extra=1)[0].cpu()
    want = plain.routed_experts(x.double(), {plain_names[local]: tensor.double() for local, tensor in tensors.items()},
                                {"router": {"experts": experts, "top": top}, "shared": {"ff": shared_ff}}, chosen)
    terms = part.forward(on(x, dtype), defer=True)
    assert isinstance(terms, ops.TermSum)
    close(terms.sum(), want, 1e-5 if dtype == torch.float32 else 2e-2)
    close(part.forward(on(x, dtype)), want, 1e-5 if dtype == torch.float32 else 2e-2)
