"""The kernels that came with the Sorizen decoder, each alone against its plain PyTorch statement, at
sizes other than any model's: the residual streams' write, read and norm in one pass, the store
kernel of latent attention without a query latent, windows, sinks and gates in the attention kernels
over rows that are keys and values at once, the router's groups by their two best scores, the exact
GELU."""
import pytest
import torch

import kernel_references as ref
from test_gpu_kernels import _attention_case, status, tol

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def dev():
    return torch.device("cuda:0")


def close(got, want, dtype):
    torch.testing.assert_close(got, want, **(dict(rtol=1e-4, atol=2e-5) if dtype == torch.float32 else tol(dtype)))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("tokens, hidden, splits", [
    (1, 64, 1), (5, 320, 7), (9, 100, 20), (6, 37, 3), (200, 48, 1), (333, 1000, 1), (150, 1536, 1), (12, 2500, 16),
    (140, 4096, 1), (3, 5000, 2), (150, 51, 1),
])
def test_streams_write_read_and_norm(dev, dtype, streams, tokens, hidden, splits):
    """Few rows with partial sums, many rows, widths no vector fits; the first write makes the streams of one
    row, later ones work in place; a look at some rows stores nothing."""
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(1)

    def floats(*shape, scale=1.0, offset=0.0):
        return (offset + scale * torch.randn(shape, generator=gen)).to(dev)

    pending = floats(splits, tokens, hidden) if splits > 1 else floats(tokens, hidden).to(dtype)
    mix, write, read = floats(streams, streams), floats(streams), floats(streams)
    weight, bias = floats(hidden, scale=0.1, offset=1.0), floats(hidden)
    first = floats(tokens, hidden, offset=2.0)
    rows = torch.tensor([tokens - 1, 0, tokens // 2], dtype=torch.int32, device=dev)
    for centre in (True, False):
        results = []
        for fn in (ops.hyper_norm, ref.hyper_norm):
            outs = [torch.full((tokens, hidden), float("nan"), dtype=dtype, device=dev) for _ in range(3)]
            picked = torch.full((3, hidden), float("nan"), dtype=dtype, device=dev)
            made = torch.full((streams, tokens, hidden), float("nan"), device=dev)
            eps = 1e-5
            fn(None, first, streams, None, read, None, weight, bias, centre, eps, outs[0])
            fn(pending, first, streams, (mix, write), read, made, weight, bias if centre else None, centre, eps, outs[1])
            after_first = made.clone()
            fn(pending, made, streams, (mix, write), None, None, weight, bias, centre, eps, picked, rows)
            assert torch.equal(made, after_first)
            fn(pending, made, streams, (mix, write), read, made, weight, bias, centre, eps, outs[2])
            results.append((*outs, picked, after_first, made))
        for got, want in zip(*results):
            close(got, want, got.dtype if got.dtype == torch.bfloat16 else torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, hidden", [(7, 64), (300, 768), (5, 33)])
def test_layer_norm_on_one_plain_stream(dev, dtype, tokens, hidden):
    """The norm part as a model with one stream uses it: the pending output is added to the residual."""
    from einf_b200.config.specs import PartSpec
    from einf_b200.parts.base import Runtime, build_part

    gen = torch.Generator().manual_seed(2)
    w, b = 1 + 0.1 * torch.randn(hidden, generator=gen), torch.randn(hidden, generator=gen)
    norm = build_part("norm", PartSpec("layernorm", {"size": hidden, "eps": 1e-5}), {"weight": w, "bias": b},
                      Runtime(dtype, dev))
    residual = (3 + torch.randn((tokens, hidden), generator=gen)).to(dev)
    pending = torch.randn((tokens, hidden), generator=gen).to(dtype).to(dev)
    total = residual + pending.float()
    want = torch.nn.functional.layer_norm(total, (hidden,), w.to(dev), b.to(dev), 1e-5)
    rows = torch.tensor([tokens - 1, 1], dtype=torch.int32, device=dev)
    before = residual.clone()
    close(norm.forward(pending, residual, rows=rows), want[rows.long()].to(dtype), dtype)
    assert torch.equal(residual, before)
    close(norm.forward(pending, residual), want.to(dtype), dtype)
    close(residual, total, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, rot, rank, row, interleaved, gated", [
    (4, 16, 8, 24, 32, True, True), (3, 12, 4, 20, 24, True, False), (6, 32, 16, 40, 64, False, True),
    (1, 8, 2, 8, 10, True, True), (12, 64, 32, 96, 128, True, False), (16, 128, 64, 512, 576, True, True),
])
@pytest.mark.parametrize("tokens, splits", [(9, 1), (9, 5), (310, 1)])
def test_latent_store_without_a_query_latent(dev, dtype, heads, dim, rot, rank, row, interleaved, gated, tokens, splits):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(3)
    page, pages = 4, 90
    width = rank + rot + heads * (dim + rot) + (heads if gated else 0) + 3       # three elements no one looks at
    if splits == 1:
        product = torch.randn((tokens, width), generator=gen).to(dtype).to(dev)
    else:
        product = torch.randn((splits, tokens, width), generator=gen).to(dev)
    slots = torch.randperm(page * pages, generator=gen)[:tokens].to(torch.int32)
    slots[2] = -1
    slots = slots.to(dev)
    positions = torch.randint(0, 3000, (tokens,), generator=gen).to(torch.int32).to(dev)
    inv_freq = (5000.0 ** (-torch.arange(rot // 2) / (rot // 2))).float().to(dev)
    norm = (1 + 0.1 * torch.randn(rank, generator=gen)).to(dev)
    for copied in (True, False):
        results = []
        st = status(dev)
        for fn in (ops.latent_qkv_store, ref.latent_qkv_store):
            plain = torch.zeros((tokens, heads, dim), dtype=dtype, device=dev) if copied else None
            full = torch.full((tokens, heads, row), 7.0, dtype=dtype, device=dev)
            full[:, :, rank:] = float("nan")                # all of it is written
            gate = torch.zeros((tokens, heads), device=dev) if gated else None
            cache = torch.full((pages, 1, page, row), 5.0, dtype=dtype, device=dev)
            fn(product, rank, rot, norm, 1e-5, positions, inv_freq, interleaved, 1.21, slots, plain, full, gate, cache, st,
               dim)
            results.append([t for t in (plain, full, gate, cache) if t is not None])
        assert int(st) == 0
        for got, want in zip(*results):
            close(got, want, got.dtype if got.dtype == torch.bfloat16 else torch.float32)
        assert bool((results[0][1 if copied else 0][:, :, :rank] == 7.0).all())      # the absorbed part is someone else's
    slots[1] = page * pages + 3                             # beyond the pool: reported, not written
    ops.latent_qkv_store(product, rank, rot, norm, 1e-5, positions, inv_freq, interleaved, 1.0, slots, None, full, gate,
                         cache, st, dim)
    assert int(st) == ops.STATUS_BAD_PAGE


def sink_and_gate(dev, heads, tokens):
    gen = torch.Generator().manual_seed(4)
    sink = (torch.randn(heads, generator=gen) * 3).to(dev)
    sink[0], sink[-1] = 40.0, -40.0          # nearly all of the weight; as good as absent
    return sink, torch.rand((tokens, heads), generator=gen).to(dev)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, rank, rot, page_size", [(3, 24, 8, 4), (18, 96, 48, 16), (5, 512, 64, 16), (1, 9, 2, 8)])
@pytest.mark.parametrize("window", [None, 1, 33, 150])
def test_shared_row_decode_with_window_sink_and_gate(dev, dtype, heads, rank, rot, page_size, window):
    from einf_b200 import ops

    row = rank + rot
    requests = [(0, 1), (page_size * 4 - 1, 1), (31, 1), (32, 1), (33, 1), (149, 1), (150, 1), (700, 1)]
    (q, k, _, table, seq, pos), _, _ = _attention_case(dev, dtype, heads, 1, row, page_size, requests, window)
    sink, gate = sink_and_gate(dev, heads, q.shape[0])
    scale = 2.0 * row ** -0.5
    for splits in (1, 3, 8):
        for s, g in ((sink, None), (None, gate), (sink, gate)):
            out = torch.full((q.shape[0], heads, rank), float("nan"), dtype=dtype, device=dev)
            want = torch.empty_like(out)
            st = status(dev)
            ops.latent_decode_attention(q, k, table, seq, pos, out, scale, splits, st, window, s, g)
            ref.latent_decode_attention(q, k, table, seq, pos, want, scale, splits, st, window, s, g)
            assert int(st) == 0
            close(out, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, rank, rot", [(3, 24, 8), (4, 512, 64)])
@pytest.mark.parametrize("window", [None, 5])
def test_general_attention_with_a_gate(dev, dtype, heads, rank, rot, window):
    from einf_b200 import ops

    requests = [(0, 1), (0, 8), (3, 6), (15, 6), (70, 1), (0, 37)]
    (q, k, _, table, seq, pos), scale, _ = _attention_case(dev, dtype, heads, 1, rank + rot, 4, requests, window)
    sink, gate = sink_and_gate(dev, heads, q.shape[0])
    out = torch.full((q.shape[0], heads, rank), float("nan"), dtype=dtype, device=dev)
    want = torch.empty_like(out)
    st = status(dev)
    ops.paged_attention_generic(q, k, None, table, seq, pos, out, scale, window, st, values_in_keys=rank, sink=sink, gate=gate)
    ref.paged_attention_generic(q, k, None, table, seq, pos, want, scale, window, st, values_in_keys=rank, sink=sink, gate=gate)
    assert int(st) == 0
    close(out, want, dtype)


@pytest.mark.parametrize("size", [64, 128])
@pytest.mark.parametrize("heads", [1, 6, 18])
@pytest.mark.parametrize("window", [None, 40, 1000])
def test_tensor_core_attention_with_a_gate(dev, size, heads, window):
    """Row tiles alone and clusters that share one, single tokens in one cluster and in several."""
    from einf_b200 import ops

    dtype = torch.bfloat16
    requests = [(0, 130), (2100, 70), (0, 5), (1500, 1), (63, 1), (0, 1)]
    (q, k, _, table, seq, pos), scale, _ = _attention_case(dev, dtype, heads, 1, size, 16, requests, window)
    sink, gate = sink_and_gate(dev, heads, q.shape[0])
    want = torch.zeros((q.shape[0], heads, size), dtype=dtype, device=dev)
    st = status(dev)
    ref.paged_attention_generic(q, k, k, table, seq, pos, want, scale, window, st, sink=sink, gate=gate)
    tiles, token = [], 0
    singles = []
    for r, (start, n) in enumerate(requests):
        if n == 1:
            singles.append(token)
        else:
            for at in range(0, n, 128):
                tiles.append([r, token + at, min(128, n - at), start + at])
        token += n
    tiles = torch.tensor(tiles, dtype=torch.int32, device=dev)
    single_tokens = torch.tensor(singles, dtype=torch.int32, device=dev)
    for cluster in (1, 4):
        out = torch.zeros_like(want)
        ops.paged_prefill_attention(q, k, k, table, tiles, out, scale, window, st, prefill_cluster=cluster, sink=sink,
                                    gate=gate)
        for clusters, splits in ((1, 1), (4, 1), (2, 2)):
            ops.paged_decode_attention_tcgen05(q, k, k, table, seq, pos, out, scale, window, clusters, st, single_tokens,
                                               splits, sink=sink, gate=gate)
            torch.testing.assert_close(out, want, rtol=3e-2, atol=2e-2)
    assert int(st) == 0


@pytest.mark.parametrize("experts, top, groups", [
    (15, 2, (3, 2)), (12, 4, (4, 2)), (9, 3, (3, 1)), (8, 8, (4, 4)), (6, 2, (6, 3)), (5, 2, None), (1, 1, (1, 1)),
    (160, 8, (40, 5)), (64, 6, (2, 1)),
])
@pytest.mark.parametrize("score", ["sigmoid", "softmax"])
@pytest.mark.parametrize("corrected", [False, True])
def test_router_with_groups_by_their_two_best(dev, experts, top, groups, score, corrected):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(5)
    logits = (torch.randn((43, experts), generator=gen) * 2).to(dev)
    correction = (torch.randn(experts, generator=gen) * 0.2).to(dev) if corrected else None
    results = []
    for fn in (ops.router_topk, ref.router_topk):
        ids = torch.zeros((43, top), dtype=torch.int32, device=dev)
        weights = torch.zeros((43, top), dtype=torch.float32, device=dev)
        fn(logits, top, score, True, ids, weights, experts, correction, groups, group_best=2, renormalise_eps=0.25,
           weight_scale=1.75)
        results.append((ids, weights))
    assert torch.equal(results[0][0], results[1][0])
    torch.testing.assert_close(results[0][1], results[1][1], rtol=1e-5, atol=1e-7)
    # written out for a few rows
    scores = (torch.softmax(logits, dim=-1) if score == "softmax" else torch.sigmoid(logits)).double().cpu()
    choice = scores + (0 if correction is None else correction.double().cpu())
    for t in range(6):
        chosen = results[0][0][t].tolist()
        if groups is not None:
            per = experts // groups[0]
            pairs = [sum(sorted(choice[t, g * per:(g + 1) * per].tolist())[-2:]) for g in range(groups[0])]
            kept = set(sorted(range(groups[0]), key=lambda g: -pairs[g])[:groups[1]])
            assert {e // per for e in chosen} <= kept
        total = sum(float(scores[t, e]) for e in chosen) + 0.25
        for j, e in enumerate(chosen):
            assert float(results[0][1][t, j]) == pytest.approx(1.75 * float(scores[t, e]) / total, rel=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("splits", [1, 3])
def test_exact_gelu(dev, dtype, splits):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(6)
    x = (3 * torch.randn((splits, 11, 56), generator=gen)).to(dev)
    x = x if splits > 1 else x[0].to(dtype)
    out = torch.empty((11, 56), dtype=dtype, device=dev)
    ops.activation(x, out, "gelu")
    z = x.double().sum(0) if splits > 1 else x.double()
    want = torch.nn.functional.gelu(z)
    close(out, want.to(dtype), dtype)


@pytest.mark.parametrize("heads, rank, rot, row", [
    (1, 50, 14, 64), (7, 136, 24, 192), (18, 300, 20, 320), (12, 512, 64, 576), (130, 96, 32, 128), (5, 400, 48, 448),
    (3, 600, 40, 640),
])
@pytest.mark.parametrize("page_size", [8, 16, 64])
@pytest.mark.parametrize("window", [None, 1, 40, 1000])
def test_latent_attention_on_the_tensor_cores(dev, heads, rank, rot, row, page_size, window):
    """Portions beside single tokens, rows longer than what they hold, values in one and in two parts, keys in shares."""
    from einf_b200 import ops

    dtype = torch.bfloat16
    requests = [(0, 131), (1100, 70), (0, 5), (1500, 1), (63, 1), (0, 1), (200, 2)]
    (q, k, _, table, seq, pos), _, _ = _attention_case(dev, dtype, heads, 1, row, page_size, requests, window)
    q[:, :, rank + rot:] = 0
    k[..., rank + rot:] = 0
    sink, gate = sink_and_gate(dev, heads, q.shape[0])
    scale = 2.0 * (rank + rot) ** -0.5
    tiles, singles, token = [], [], 0
    for r, (start, n) in enumerate(requests):
        if n == 1:
            singles.append(token)
        for at in range(0, n if n > 1 else 0, 128):
            tiles.append([r, token + at, min(128, n - at), start + at])
        token += n
    tiles = torch.tensor(tiles, dtype=torch.int32, device=dev)
    listed = torch.tensor(singles, dtype=torch.int32, device=dev)
    for s, g in ((None, None), (sink, gate)):
        st = status(dev)
        want = torch.zeros((q.shape[0], heads, rank), dtype=dtype, device=dev)
        ref.paged_attention_generic(q, k, None, table, seq, pos, want, scale, window, st, values_in_keys=rank, sink=s, gate=g)
        for longest in (100, 1501):           # the longest context sets the number of shares
            out = torch.full((q.shape[0], heads, rank), float("nan"), dtype=dtype, device=dev)
            ops.latent_attention(q, k, table, seq, pos, tiles, listed, len(singles), out, scale, window, st,
                                 max_context=longest, sink=s, gate=g)
            torch.testing.assert_close(out, want, rtol=3e-2, atol=2e-2)
        # the same single tokens alone, as a decode step has them
        picked = [t[listed.long()].contiguous() for t in (q, seq, pos)]
        alone = torch.full((len(singles), heads, rank), float("nan"), dtype=dtype, device=dev)
        ops.latent_attention(picked[0], k, table, picked[1], picked[2], None, None, len(singles), alone, scale, window, st,
                             max_context=1501, sink=s, gate=None if g is None else g[listed.long()].contiguous())
        assert torch.equal(alone, out[listed.long()])
        assert int(st) == 0


def test_latent_attention_reports_a_page_outside_the_pool(dev):
    from einf_b200 import ops

    (q, k, _, table, seq, pos), scale, _ = _attention_case(dev, torch.bfloat16, 4, 1, 192, 16, [(0, 60)], None)
    table[0, 2] = k.shape[0] + 5              # reported, not read
    st = status(dev)
    out = torch.zeros((60, 4, 128), dtype=torch.bfloat16, device=dev)
    tiles = torch.tensor([[0, 0, 60, 0]], dtype=torch.int32, device=dev)
    ops.latent_attention(q, k, table, seq, pos, tiles, None, 0, out, scale, None, st)
    assert int(st) == ops.STATUS_BAD_PAGE and torch.isfinite(out).all()
