"""The kernels that came with the Pugadra decoder, each alone against its plain PyTorch statement, at
sizes other than any model's: the store kernel with its convolution (head by head and in 16-byte pieces),
the stream's norms in front of and behind a sublayer, the token input's gate, the clamped gate, the router's bias, an output gate per element in the attention kernels."""
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


def conv_case(dev, dtype, heads, kv_heads, size, vsize, taps, portions, splits, gated, pairs, seed=3):
    """``portions``: tokens that every request brings; every second request goes on from an earlier step."""
    gen = torch.Generator().manual_seed(seed)
    tokens, page, pages = sum(portions), 8, sum(portions) // 8 + 12
    channels = (heads + kv_heads) * size + kv_heads * vsize
    width = channels + (heads * vsize if gated else 0)
    product = torch.randn((splits, tokens, width), generator=gen)
    product = product.to(dev) if splits > 1 else product[0].to(dtype).to(dev)
    starts = [0]
    for n in portions:
        starts.append(starts[-1] + n)
    slots = torch.randperm(page * pages, generator=gen)[:tokens].to(torch.int32)
    if tokens > 2:
        slots[2] = -1
    requests = len(portions)
    state_slots = torch.randperm(requests + 2, generator=gen)[:requests].to(torch.int32)
    state = torch.randn((requests + 2, (taps - 1) * channels + 5), generator=gen)
    for r in range(0, requests, 2):
        state[int(state_slots[r]), :(taps - 1) * channels] = 0.0         # starts in this step
    if requests > 3:
        state_slots[3] = -1
    return dict(
        product=product, bias=torch.randn(channels, generator=gen).to(dev),
        weight=(torch.randn((channels, taps), generator=gen) + 0.3).to(dev), state=state.to(dev),
        seq=torch.repeat_interleave(torch.arange(requests), torch.tensor(portions)).to(torch.int32).to(dev),
        q_start=torch.tensor(starts, dtype=torch.int32, device=dev), state_slots=state_slots.to(dev), slots=slots.to(dev),
        positions=torch.randint(0, 3000, (tokens,), generator=gen).to(torch.int32).to(dev),
        inv_freq=(4000.0 ** (-torch.arange(pairs) / max(pairs, 1))).float().to(dev),
        channels=channels, tokens=tokens, page=page, pages=pages)


def run_conv(fn, c, dev, dtype, heads, kv_heads, size, vsize, taps, interleaved, gated, single, bias=True, weight=True):
    q = torch.full((c["tokens"], heads, size), float("nan"), dtype=dtype, device=dev)
    groups = max(kv_heads, 1)
    k = torch.full((c["pages"], groups, c["page"], size), 5.0, dtype=dtype, device=dev)
    v = torch.full((c["pages"], groups, c["page"], vsize), 5.0, dtype=dtype, device=dev)
    gate = torch.full((c["tokens"], heads * vsize), float("nan"), dtype=dtype, device=dev) if gated else None
    state = c["state"].clone()
    rows = None
    if taps > 1 and weight:
        rows = state[:, :(taps - 1) * c["channels"]].unflatten(1, (taps - 1, c["channels"]))
    st = status(dev)
    fn(c["product"], c["bias"] if bias else None, c["weight"] if weight else None, rows, c["seq"], c["q_start"],
       c["state_slots"], c["slots"] if kv_heads else None, q, k if kv_heads else None, v if kv_heads else None, heads,
       kv_heads, size, vsize, st, positions=c["positions"], inv_freq=c["inv_freq"], interleaved=interleaved,
       gate_out=gate, single_tokens=single)
    assert int(st) == 0
    return [t for t in (q, k, v, gate, state) if t is not None]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, size, vsize, pairs, interleaved", [
    (4, 2, 16, 24, 4, True), (3, 1, 10, 6, 5, True), (5, 0, 32, 16, 16, False), (2, 2, 64, 64, 32, True),
    (14, 2, 64, 64, 32, True), (1, 1, 128, 256, 0, False), (6, 3, 40, 8, 12, True), (20, 4, 128, 128, 64, True),
])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("portions, splits", [
    ((1, 2, 9, 3, 1, 5), 1), ((1, 2, 9, 3, 1, 5), 3), ((50, 1, 2, 3, 40, 7, 8, 1, 1, 100), 1),
])
def test_convolve_rotate_and_store(dev, dtype, heads, kv_heads, size, vsize, pairs, interleaved, taps, portions, splits):
    """Portions down to a single token, requests that start beside such that go on, a request without a state slot and
    a token that is not cached; long steps of bfloat16 rows take the kernel of 16-byte pieces."""
    from einf_b200 import ops

    gated = splits > 1
    c = conv_case(dev, dtype, heads, kv_heads, size, vsize, taps, portions, splits, gated, pairs)
    args = (c, dev, dtype, heads, kv_heads, size, vsize, taps, interleaved, gated, False)
    for got, want in zip(run_conv(ops.qkv_conv_store, *args), run_conv(ref.qkv_conv_store, *args)):
        close(got, want, got.dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 9])
@pytest.mark.parametrize("splits, gated", [(1, False), (12, True), (20, False)])
def test_single_tokens_move_the_state_on_in_one_launch(dev, dtype, taps, splits, gated):
    from einf_b200 import ops

    heads, kv_heads, size, vsize = 6, 2, 32, 48
    c = conv_case(dev, dtype, heads, kv_heads, size, vsize, taps, (1,) * 7, splits, gated, 12)
    args = (c, dev, dtype, heads, kv_heads, size, vsize, taps, True, gated, True)
    before = ops.launch_count
    got = run_conv(ops.qkv_conv_store, *args)
    assert ops.launch_count == before + 1
    for mine, want in zip(got, run_conv(ref.qkv_conv_store, *args)):
        close(mine, want, mine.dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_store_without_its_options(dev, dtype):
    """No bias, no convolution (an output gate alone), columns beside the gate left where they are; a slot beyond the
    pool is reported and not written."""
    from einf_b200 import ops

    heads, kv_heads, size, vsize = 4, 2, 16, 16
    c = conv_case(dev, dtype, heads, kv_heads, size, vsize, 1, (40, 3), 1, True, 8)
    args = (c, dev, dtype, heads, kv_heads, size, vsize, 1, True, False, False, False, False)
    for got, want in zip(run_conv(ops.qkv_conv_store, *args), run_conv(ref.qkv_conv_store, *args)):
        close(got, want, got.dtype)
    c["slots"][1] = c["page"] * c["pages"] + 2
    q = torch.empty((43, heads, size), dtype=dtype, device=dev)
    k = torch.full((c["pages"], kv_heads, c["page"], size), 5.0, dtype=dtype, device=dev)
    st = status(dev)
    ops.qkv_conv_store(c["product"], None, None, None, c["seq"], c["q_start"], c["state_slots"], c["slots"], q, k, k.clone(),
                       heads, kv_heads, size, vsize, st, positions=c["positions"], inv_freq=c["inv_freq"], interleaved=True)
    assert int(st) == ops.STATUS_BAD_PAGE


def test_a_portions_cut_changes_nothing(dev):
    """The same forty tokens as one portion, and as portions of eight kinds one after the other: the same bits in float32."""
    from einf_b200 import ops

    heads, kv_heads, size, vsize, taps = 3, 1, 16, 16, 4
    c = conv_case(dev, torch.float32, heads, kv_heads, size, vsize, taps, (40,), 1, False, 8)
    c["slots"] = torch.arange(40, dtype=torch.int32, device=dev)
    c["state_slots"] = torch.zeros(1, dtype=torch.int32, device=dev)
    c["state"].zero_()
    whole = run_conv(ops.qkv_conv_store, c, dev, torch.float32, heads, kv_heads, size, vsize, taps, True, False, False)
    state = torch.zeros_like(c["state"])
    rows = state[:, :(taps - 1) * c["channels"]].unflatten(1, (taps - 1, c["channels"]))
    q, k, v = torch.zeros_like(whole[0]), torch.full_like(whole[1], 5.0), torch.full_like(whole[2], 5.0)
    at, st = 0, status(dev)
    for n in (1, 2, 3, 2, 1, 1, 9, 21):
        part = slice(at, at + n)
        ops.qkv_conv_store(c["product"][part].contiguous(), c["bias"], c["weight"], rows, c["seq"][part].contiguous(),
                           torch.tensor([0, n], dtype=torch.int32, device=dev), c["state_slots"], c["slots"][part].contiguous(),
                           q[part], k, v, heads, kv_heads, size, vsize, st, positions=c["positions"][part].contiguous(),
                           inv_freq=c["inv_freq"], interleaved=True, single_tokens=n == 1)
        at += n
    assert torch.equal(q, whole[0]) and torch.equal(k, whole[1]) and torch.equal(v, whole[2])
    assert torch.equal(state[0, :(taps - 1) * c["channels"]], whole[3][0, :(taps - 1) * c["channels"]])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, hidden, splits, two", [
    (1, 64, 1, False), (5, 320, 7, False), (9, 100, 20, True), (6, 37, 3, False), (300, 48, 1, False), (333, 1000, 1, False),
    (290, 1536, 1, True), (12, 2500, 16, False), (260, 2048, 1, False), (300, 3584, 1, False), (3, 9000, 2, False),
    (270, 51, 1, False), (2, 1023, 4, True), (7, 5120, 13, False),
])
def test_norms_behind_and_in_front_of_a_sublayer(dev, dtype, tokens, hidden, splits, two):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(1)

    def floats(*shape, scale=1.0, offset=0.0):
        return (offset + scale * torch.randn(shape, generator=gen)).to(dev)

    pending = [floats(splits, tokens, hidden) if splits > 1 else floats(tokens, hidden).to(dtype)]
    if two:
        pending.append(floats(tokens, hidden))
    post, norm = (floats(hidden, scale=0.3, offset=1.0), 1e-5), (floats(hidden, scale=0.3, offset=1.0), 1e-6)
    first = floats(tokens, hidden, offset=0.5)
    for behind in (post, None):
        for ahead, stored in ((norm, True), (None, True), (None, False)):
            for terms in (pending, None):
                results = []
                for fn in (ops.stream_norm, ref.stream_norm):
                    residual = first.clone()
                    out = torch.full((tokens, hidden), float("nan"), dtype=dtype, device=dev) if stored else None
                    fn(terms, 0.7, behind, residual, ahead, out)
                    results.append([t for t in (residual, out) if t is not None])
                for got, want in zip(*results):
                    close(got, want, got.dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, side, splits", [(1, 16, 1), (300, 64, 1), (9, 7, 5)])
def test_the_token_inputs_gate(dev, dtype, tokens, side, splits):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(3)
    product = (2 * torch.randn((splits, tokens, side), generator=gen)).to(dev)
    product = product if splits > 1 else product[0].to(dtype)
    table = torch.randn((30, side), generator=gen).to(dtype).to(dev)
    ids = torch.randint(0, 30, (tokens,), generator=gen).to(torch.int32).to(dev)
    results = []
    for fn in (ops.side_gate, ref.side_gate):
        out = torch.full((tokens, side), float("nan"), dtype=dtype, device=dev)
        fn(product, table, ids, out)
        results.append(out)
    close(*results, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, inter, splits", [(1, 8, 1), (9, 96, 4), (300, 1000, 1), (5, 37, 1), (7, 64, 20)])
@pytest.mark.parametrize("limit, slope, shift", [(0.7, 1.702, 1.0), (7.0, 1.0, 0.0), (1.5, 3.0, -0.5)])
def test_the_clamped_gate(dev, dtype, tokens, inter, splits, limit, slope, shift):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(4)
    x = (3 * torch.randn((splits, tokens, 2 * inter), generator=gen)).to(dev)
    x = x if splits > 1 else x[0].to(dtype)
    results = []
    for fn in (ops.act_mul, ref.act_mul):
        out = torch.full((tokens, inter), float("nan"), dtype=dtype, device=dev)
        fn(x, out, "clamped_swish", limit=limit, slope=slope, up_shift=shift)
        results.append(out)
    close(*results, dtype)
    z = x.double().sum(0) if splits > 1 else x.double()
    g, u = torch.clamp(z[:, :inter], max=limit), torch.clamp(z[:, inter:], -limit, limit)
    close(results[0], (g * torch.sigmoid(slope * g) * (u + shift)).to(dtype), dtype)


@pytest.mark.parametrize("experts, top, splits", [(15, 3, 1), (4, 4, 5), (1, 1, 1), (160, 8, 1)])
def test_the_routers_bias_takes_part_in_choice_and_weights(dev, experts, top, splits):
    from einf_b200 import ops

    gen = torch.Generator().manual_seed(5)
    logits = torch.randn((splits, 43, experts), generator=gen).to(dev)
    logits = logits if splits > 1 else logits[0]
    bias = (3 * torch.randn(experts, generator=gen)).to(dev)
    ids = torch.zeros((43, top), dtype=torch.int32, device=dev)
    weights = torch.zeros((43, top), dtype=torch.float32, device=dev)
    ops.router_topk(logits, top, "softmax", True, ids, weights, experts, bias=bias)
    z = (logits.double().sum(0) if splits > 1 else logits.double()) + bias.double()
    best = torch.topk(z, top)
    assert torch.equal(ids.long(), best.indices)
    torch.testing.assert_close(weights.double(), torch.softmax(best.values, dim=-1), rtol=1e-5, atol=1e-7)


def gate_logits(dev, dtype, tokens, width, wide):
    """Logits as columns of a wider matrix, or alone."""
    gen = torch.Generator().manual_seed(6)
    whole = (2 * torch.randn((tokens, width + (24 if wide else 0)), generator=gen)).to(dtype).to(dev)
    return whole[:, whole.shape[1] - width:]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv_heads, size, vsize", [(4, 2, 16, 16), (3, 1, 10, 30), (6, 3, 64, 48)])
@pytest.mark.parametrize("window", [None, 5])
@pytest.mark.parametrize("wide", [False, True])
def test_general_attention_with_a_gate_per_element(dev, dtype, heads, kv_heads, size, vsize, window, wide):
    from einf_b200 import ops

    requests = [(0, 1), (0, 8), (3, 6), (15, 6), (70, 1), (0, 37)]
    (q, k, v, table, seq, pos), scale, _ = _attention_case(dev, dtype, heads, kv_heads, size, 4, requests, window)
    v = torch.randn((*v.shape[:3], vsize), generator=torch.Generator().manual_seed(1)).to(dtype).to(dev)
    sink = torch.zeros(heads, device=dev)
    logits = gate_logits(dev, dtype, q.shape[0], heads * vsize, wide)
    out = torch.full((q.shape[0], heads, vsize), float("nan"), dtype=dtype, device=dev)
    want = torch.empty_like(out)
    st = status(dev)
    ops.paged_attention_generic(q, k, v, table, seq, pos, out, scale, window, st, sink=sink, value_gate=logits)
    ref.paged_attention_generic(q, k, v, table, seq, pos, want, scale, window, st, sink=sink, value_gate=logits)
    assert int(st) == 0
    close(out, want, dtype)


@pytest.mark.parametrize("size", [64, 128])
@pytest.mark.parametrize("heads, kv_heads", [(1, 1), (6, 2), (18, 1)])
@pytest.mark.parametrize("window", [None, 40, 1000])
def test_tensor_core_attention_with_a_gate_per_element(dev, size, heads, kv_heads, window):
    """Row tiles alone and clusters that share one, single tokens in one cluster and in several, logits as columns of a
    wider matrix; the sink of score zero that goes with it."""
    from einf_b200 import ops

    dtype = torch.bfloat16
    requests = [(0, 130), (2100, 70), (0, 5), (1500, 1), (63, 1), (0, 1)]
    (q, k, v, table, seq, pos), scale, _ = _attention_case(dev, dtype, heads, kv_heads, size, 16, requests, window)
    sink = torch.zeros(heads, device=dev)
    logits = gate_logits(dev, dtype, q.shape[0], heads * size, True)
    want = torch.zeros((q.shape[0], heads, size), dtype=dtype, device=dev)
    st = status(dev)
    ref.paged_attention_generic(q, k, v, table, seq, pos, want, scale, window, st, sink=sink, value_gate=logits)
    tiles, token, singles = [], 0, []
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
        ops.paged_prefill_attention(q, k, v, table, tiles, out, scale, window, st, prefill_cluster=cluster, sink=sink,
                                    value_gate=logits)
        for clusters, splits in ((1, 1), (4, 1), (2, 2)):
            ops.paged_decode_attention_tcgen05(q, k, v, table, seq, pos, out, scale, window, clusters, st, single_tokens,
                                               splits, sink=sink, value_gate=logits)
            torch.testing.assert_close(out, want, rtol=3e-2, atol=2e-2)
    assert int(st) == 0
    with pytest.raises(ops.UnsupportedSize):        # the prompt kernel reads 16-byte pieces
        wider = torch.zeros((q.shape[0], heads * size + 4), dtype=dtype, device=dev)
        ops.paged_prefill_attention(q, k, v, table, tiles, out, scale, window, st, sink=sink, value_gate=wider[:, 4:])
