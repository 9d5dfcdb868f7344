"""The Sorizen decoder in the engine against the plain statement of ``sorizen_plain``.

Small configurations of their own, random weights, every position of every request compared.  The
scenarios run twice: on the CPU through the plain statements of the kernels
(``kernel_references.emulate_kernels``: what is under test then is the configuration, the weights'
names, the layers that share tensors, the residual streams, the cache plan with a page group per
window, batch packing, replay and scheduler), and, marked ``gpu``, on the kernels in float32 and
bfloat16.
"""
from __future__ import annotations

import copy
import json
import math

import numpy as np
import pytest
import torch
from safetensors.torch import save_file

import sorizen_plain
import trace_tools
from conftest import random_tokens
from kernel_references import emulate_kernels

SINK, GATE = "latent_attention", "latent_attention_2"


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, scale=1.0):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def yarn(factor, original, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def layer(kind, heads, dim, rot_dim, vdim, kv_rank, size, mlp, scale=0.3, base=100.0, scaling=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
             "rot": {"base": base, "dims": rot_dim}}
    if size is not None:
        mixer["mask"] = {"size": size}
    if scaling is not None:
        mixer["rot"]["scaling"] = scaling
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(width, vocab, layers, streams=2, scale=0.5, eps=1e-5):
    config = {"architecture": "Sorizen", "vocab": vocab, "width": width, "norm": {"eps": eps},
              "embedding": {"scale": scale}, "streams": streams, "layers": []}
    for entry in layers:
        if isinstance(entry, int):          # the tensors of that layer once more
            entry = dict(copy.deepcopy(config["layers"][entry]), weights_of=entry)
        config["layers"].append(entry)
    return config


CONFIGS = {
    # layers that differ in every size; three streams; windows that are no multiple of a page and a layer that sees
    # everything; stretched frequencies whose ramp lies inside the table, one layer without; a layer without a
    # feed-forward; two layers that run with another layer's tensors, one of them twice removed in place
    "mix": model(48, 97, [
        layer(GATE, 4, 16, 8, 12, 24, 7, dense(56), scaling=yarn(4.0, 64)),
        layer(SINK, 3, 8, 4, 20, 40, 13, moe(24, 12, 3, groups=(4, 2), scale=2.2), base=500.0, scaling=yarn(2.0, 40, 4.0, 0.5)),
        layer(SINK, 6, 8, 12, 8, 20, None, None, scale=0.5),
        1,
        layer(GATE, 2, 24, 16, 32, 32, 20, moe(32, 6, 2, groups=(2, 1), scale=1.5), base=10000.0, scaling=yarn(6.0, 900, 24.0)),
        0,
        1,
    ], streams=3, scale=0.7),
    # what the sizes above make unequal, here equal or 1: one stream, one head, one pair, a window of one key, one
    # expert, one group, groups of one expert, scales of one
    "ones": model(40, 61, [
        layer(GATE, 1, 8, 2, 8, 8, 1, moe(8, 1, 1, groups=(1, 1)), scaling=yarn(1.0, 16)),
        layer(SINK, 1, 16, 16, 16, 16, 2, moe(16, 4, 2, groups=(4, 2)), scale=1.0),
        layer(GATE, 5, 8, 8, 8, 8, 3, dense(40)),
    ], streams=1, scale=1.0, eps=1e-6),
    # no groups, no stretched frequencies, no window; four streams
    "bare": model(32, 50, [layer(SINK, 2, 16, 8, 16, 24, None, moe(24, 5, 2)),
                           layer(GATE, 2, 8, 16, 8, 16, None, dense(24))], streams=4),
    # rows that the tensor-core attention kernels take (filled up to 64 and 128), windows longer than a key tile
    "wide": model(64, 83, [
        layer(GATE, 4, 32, 16, 32, 112, 150, dense(96), scale=0.14, scaling=yarn(8.0, 256, 16.0)),
        layer(SINK, 3, 16, 8, 24, 40, 33, moe(32, 8, 2, groups=(4, 2), scale=2.0), scale=0.2),
        layer(SINK, 2, 32, 32, 64, 96, None, dense(64), scale=0.125),
    ]),
    # longer rows, sixteen and more heads
    "long_rows": model(64, 71, [
        layer(SINK, 18, 16, 16, 16, 144, 40, dense(64), scale=0.18, scaling=yarn(2.0, 128)),
        layer(GATE, 5, 32, 32, 32, 288, 70, moe(32, 4, 2, scale=1.5), scale=0.125),
    ]),
}
PAGE = {"mix": 4, "ones": 8, "bare": 16, "wide": 16, "long_rows": 16}
SINGLE = {
    # one mechanism at a time
    "sink": model(32, 50, [layer(SINK, 4, 8, 4, 8, 16, 6, None)], streams=1),
    "gate": model(32, 50, [layer(GATE, 4, 8, 4, 8, 16, 6, None)], streams=1),
    "streams": model(32, 50, [layer(GATE, 1, 8, 4, 8, 16, 50, None), layer(SINK, 1, 8, 4, 8, 16, 50, dense(32))], streams=5),
    "routed": model(32, 50, [layer(SINK, 1, 8, 4, 8, 16, 50, moe(24, 15, 3, groups=(3, 2), scale=2.0))], streams=1),
    "shared_tensors": model(32, 50, [layer(SINK, 2, 8, 4, 8, 16, 5, dense(24)), 0, 0], streams=2),
}


def every_expert(config):
    """The same sizes with a router that chooses every expert: nothing rests on a close call, which
    bfloat16 would flip within a dozen tokens."""
    config = copy.deepcopy(config)
    for entry in config["layers"]:
        mlp = entry.get("mlp")
        if mlp is not None and mlp["kind"] == "moe":
            mlp["router"]["top"] = mlp["router"]["experts"]
            if "groups" in mlp["router"]:
                mlp["router"]["groups"]["keep"] = mlp["router"]["groups"]["count"]
    return config


def write_folder(folder, config, seed, weights=None):
    folder.mkdir(parents=True, exist_ok=True)
    weights = weights if weights is not None else sorizen_plain.random_model(config, seed)
    (folder / "config.json").write_text(json.dumps(config))
    save_file({k: v.contiguous() for k, v in weights.items()}, str(folder / "model.safetensors"))
    return weights


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("sorizen")
    made = {}
    for index, (name, config) in enumerate({**CONFIGS, **SINGLE}.items()):
        made[name] = (base / name, config, write_folder(base / name, config, 70 + index))
        full = every_expert(config)
        made[name + "/all"] = (base / (name + "_all"), full, write_folder(base / (name + "_all"), full, 70 + index))
    return made


CLOSE_CALL = 2e-4      # a router's margin below which a lower precision may choose otherwise


def expected_rows(config, weights, requests):
    """The plain logits of every position, and per request the first position whose router came within
    ``CLOSE_CALL`` of another choice (from there on a 32-bit run may differ by a choice)."""
    out, sure = {}, {}
    routed = sum(1 for entry in config["layers"] if (entry.get("mlp") or {}).get("kind") == "moe")
    for name, tokens in requests.items():
        margins = []
        logits, _ = sorizen_plain.forward(config, weights, tokens, margins=margins)
        for position in range(len(tokens)):
            out[(name, position)] = logits[position].float().numpy()
        sure[name] = len(tokens)
        if routed:
            close = np.nonzero(np.array(margins).reshape(routed, len(tokens)).min(axis=0) < CLOSE_CALL)[0]
            if close.size:
                sure[name] = int(close[0])
    return out, sure


def make_requests(config, lengths, seed=0):
    return {f"r{i}": random_tokens(config["vocab"], n, seed * 100 + i) for i, n in enumerate(lengths)}


def row_errors(rows, expected):
    """The error of every row (mean taken off, root mean square) against the size of the logits."""
    assert set(rows) == set(expected)
    size = math.sqrt(float(np.mean([np.var(v) for v in expected.values()])))
    errors = {}
    for key in sorted(expected):
        assert np.isfinite(rows[key]).all(), f"first wrong token: {key}"
        difference = rows[key] - expected[key]
        errors[key] = float(np.sqrt(np.mean((difference - difference.mean()) ** 2))) / size
    return errors


def conditioning(config, weights, requests, expected):
    """How far rounding alone moves every row: the plain statement in float32 against itself in float64."""
    rows = {}
    for name, tokens in requests.items():
        logits, _ = sorizen_plain.forward(config, weights, tokens, dtype=torch.float32)
        for position in range(len(tokens)):
            rows[(name, position)] = logits[position].numpy()
    return row_errors(rows, expected)


def check(rows, expected, dtype, sure=None, plain32=None, whole=None, what=""):
    """float32: every row within 2e-5 plus three times what the plain statement in float32 loses there
    (1e-4 where that is not given); rows from a request's first close call of a router on are left out.
    bfloat16 rounds 65,536 times coarser, and single rows of a narrow model with random weights move by
    tens of percent, so there the rows are held as a whole: half of them within 0.02 and nine in ten
    within 0.06 of the plain statement, and the same against the rows that the whole prompts gave
    (``whole``), from which a schedule differs only by the order of additions."""
    errors = row_errors(rows, expected)
    if dtype == "float32":
        for key, error in errors.items():
            if sure is not None and key[1] >= sure[key[0]]:
                continue
            limit = 1e-4 if plain32 is None else 2e-5 + 3.0 * plain32[key]
            assert error < limit, f"{what}: first wrong token: {key}, error {error:.2e}, limit {limit:.2e}"
        return
    for against, values in (("plain", errors), ("whole", row_errors(rows, whole) if whole is not None else None)):
        if values is not None:
            values = np.array(list(values.values()))
            assert float(np.median(values)) < 0.02 and float(np.quantile(values, 0.9)) < 0.06, \
                f"{what} against {against}: median {np.median(values):.2e}, nine in ten {np.quantile(values, 0.9):.2e}"


def replay_modes(folder, config, weights, page, dtype, device, lengths=(1, 5, 9, 23, 37, 50)):
    from einf_b200.engine.replay import TraceReplayer

    requests = make_requests(config, lengths)
    expected, sure = expected_rows(config, weights, requests)
    plain32 = conditioning(config, weights, requests, expected) if dtype == "float32" else None
    mixed_steps, most = trace_tools.mixed(requests, seed=3, page_round=page)
    room = -(-max(lengths) // 64) * 64
    traces = {
        "whole": (trace_tools.whole(requests), room),
        "tail": (trace_tools.last_one_by_one(requests, tail=12), room),
        "portions": (trace_tools.in_portions(requests), room),
        "mixed": (mixed_steps, most),
    }
    whole = None
    for mode, (steps, max_tokens) in traces.items():
        replayer = TraceReplayer(folder, dtype, max_tokens, block_len=page, device=device, max_requests=4)
        rows = trace_tools.run_steps(replayer, steps)
        check(rows, expected, dtype, sure, plain32, whole, mode)
        whole = rows if mode == "whole" else whole
        for group in range(replayer.manager.num_groups):
            assert replayer.manager.free_pages(group) == replayer.manager.group(group).num_pages, mode
        replayer.manager.check_invariants()


def for_dtype(folders, name, dtype):
    """bfloat16 runs the variant whose routers choose every expert."""
    return folders[name + "/all"] if dtype == "bfloat16" else folders[name]


# ---------------------------------------------------------------------------
# the configuration and the weights' names
def test_configuration_names_every_tensor_of_the_design(folders):
    from einf_b200.config import SorizenConfig, load_config
    from einf_b200.parts.model import expected_tensors

    for name, (folder, config, weights) in folders.items():
        loaded = load_config(folder)
        assert isinstance(loaded, SorizenConfig)
        expected, optional = expected_tensors(loaded.model_spec())
        assert set(expected) == set(weights) and not optional, name
        for key, spec in expected.items():
            assert tuple(spec.shape) == tuple(weights[key].shape), key


def test_layers_that_share_tensors_keep_caches_of_their_own(folders):
    from einf_b200.config import load_config
    from einf_b200.config.engine import EngineConfig
    from einf_b200.engine.runner import ModelRunner

    folder, config, _ = folders["mix"]
    spec = load_config(folder).model_spec()
    assert len(spec.layers) == 4 and spec.streams == 3
    assert [entry.layer for entry in spec.schedule] == [0, 1, 2, 1, 3, 0, 1]
    with emulate_kernels():
        runner = ModelRunner.from_folder(folder, EngineConfig(dtype="float32", block_len=4, num_blocks=32, device="cpu",
                                                              max_requests=3, use_cuda_graphs=False))
    plan = runner.model.cache_plan
    assert all(entry.owner == index for index, entry in enumerate(plan.entries))
    assert plan.group_windows == (7, 13, None, 20) and not plan.has_state
    assert [entry.group for entry in plan.entries] == [0, 1, 2, 1, 3, 0, 1]
    pointers = {view.k.data_ptr() for view in runner.storage.views}
    assert len(pointers) == len(config["layers"])
    assert all(view.v is None or view.v.numel() == 0 for view in runner.storage.views)     # one row is key and value


def test_configuration_refuses_what_the_design_does_not_have():
    from einf_b200.config import ConfigError, config_from_dict

    good = CONFIGS["mix"]
    config_from_dict(good)

    def broken(change):
        data = json.loads(json.dumps(good))
        change(data)
        with pytest.raises(ConfigError):
            config_from_dict(data)

    broken(lambda d: d["layers"][0].update(type="attention"))
    broken(lambda d: d["layers"][0]["mixer"].pop("kv_rank"))
    broken(lambda d: d["layers"][0]["mixer"].pop("rot"))
    broken(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=4))              # the whole part is rotated
    broken(lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"))
    broken(lambda d: d["layers"][0]["mixer"]["mask"].update(size=0))
    broken(lambda d: d["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda d: d["layers"][1]["mlp"]["router"].update(top=7))              # two groups of three can be chosen from
    broken(lambda d: d["layers"][1]["mlp"]["router"]["groups"].update(count=5))
    broken(lambda d: d["layers"][3].update(weights_of=9))
    broken(lambda d: d["layers"][3].update(weights_of=3))                        # itself
    broken(lambda d: d["layers"][3].update(weights_of=2))                        # an entry that differs
    broken(lambda d: d.update(streams=0))
    broken(lambda d: d["norm"].update(eps=0))
    broken(lambda d: d.pop("embedding"))
    broken(lambda d: d.pop("vocab"))


def test_random_weights_mode_writes_a_folder_the_loader_takes(tmp_path):
    from einf_b200.config import config_from_dict, load_config
    from einf_b200.parts.model import expected_tensors
    from einf_b200.weights import load_tensors, write_random_model

    folder = write_random_model(tmp_path / "m", config_from_dict(CONFIGS["mix"]), seed=4)
    config = load_config(folder)
    expected, optional = expected_tensors(config.model_spec())
    tensors = load_tensors(folder, expected, optional=optional)
    assert set(tensors) == set(expected)
    assert abs(float(tensors["l0.hc1.in"].float().sum()) - 1.0) < 0.7            # near the mean of the streams
    assert float((tensors["l0.hc1.mix"].float() - torch.eye(3)).abs().max()) < 1.0


# ---------------------------------------------------------------------------
# the plain statement's own mechanisms against closed forms
def test_the_plain_router_opens_the_groups_with_the_best_pairs():
    scores = torch.tensor([0.9, 0.1, 0.1, 0.6, 0.6, 0.1, 0.5, 0.1, 0.58], dtype=torch.float64)
    # pairs: 1.0, 1.2, 1.08: the group of the largest single score is the one left out
    assert sorted(sorizen_plain.route(scores, 3, {"count": 3, "keep": 2})) == [3, 4, 8]
    assert sorizen_plain.route(scores, 2) == [0, 3] or sorizen_plain.route(scores, 2) == [0, 4]
    # a group of one counts by its one member
    assert sorizen_plain.route(scores[:3], 1, {"count": 3, "keep": 1}) == [0]


def test_the_plain_frequencies_between_kept_and_stretched():
    rot = {"base": 10000.0, "dims": 32, "scaling": yarn(4.0, 2048, 32.0, 1.0)}
    table, amplitude = sorizen_plain.rotation_table(rot)
    plain = [10000.0 ** (-2 * i / 32) for i in range(16)]
    assert amplitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert table[0] == plain[0]                                          # many turns: as it was
    assert table[-1] == pytest.approx(plain[-1] / 4.0)                   # less than one turn: stretched
    shares = [(f - p / 4) / (p - p / 4) for f, p in zip(table, plain)]
    assert all(a >= b - 1e-12 for a, b in zip(shares, shares[1:])) and any(0.01 < s < 0.99 for s in shares)
    # a pair that turns exactly t times over the original length lies at dim(t)
    turns = 2048 / (2 * math.pi) * plain[5]
    assert 32 * math.log(2048 / (2 * math.pi * turns)) / (2 * math.log(10000.0)) == pytest.approx(5.0)


@pytest.mark.parametrize("dims,base,scaling", [(32, 10000.0, yarn(4.0, 2048, 32.0, 1.0)), (8, 500.0, yarn(2.0, 40, 4.0, 0.5)),
                                               (2, 100.0, yarn(1.0, 16)), (16, 1e6, yarn(8.0, 100000, 1.0, 1.0)),
                                               (16, 50.0, yarn(3.0, 4, 64.0, 0.01)), (12, 100.0, None)])
def test_the_engines_frequency_table(dims, base, scaling):
    from einf_b200.config.specs import PartSpec
    from einf_b200.parts.base import Runtime, build_part

    runtime = Runtime(torch.float32, torch.device("cpu"))
    part = build_part("position", PartSpec("rope", {
        "rotary_dim": dims, "theta": base, "layout": "interleaved",
        "scaling": None if scaling is None else dict(scaling, kind="yarn")}), {}, runtime)
    table, amplitude = sorizen_plain.rotation_table({"dims": dims, "base": base, "scaling": scaling})
    assert torch.allclose(part.inv_freq.double(), torch.tensor(table, dtype=torch.float64), rtol=2e-7, atol=0)
    assert part.amplitude == pytest.approx(amplitude)


# ---------------------------------------------------------------------------
# the engine on the plain statements of the kernels (CPU)
@pytest.fixture()
def emulated():
    with emulate_kernels():
        yield


@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone_emulated(name, folders, emulated):
    folder, config, weights = folders[name]
    replay_modes(folder, config, weights, 4, "float32", "cpu", lengths=(1, 6, 19))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_replay_modes_emulated(name, folders, emulated):
    folder, config, weights = folders[name]
    replay_modes(folder, config, weights, PAGE[name], "float32", "cpu", lengths=(1, 5, 9, 23, 37))


def test_the_streams_sum_after_every_layer_emulated(folders, emulated):
    """The streams as the engine holds them, with what is pending, against the plain statement's."""
    from einf_b200.engine.replay import TraceReplayer

    folder, config, weights = folders["mix"]
    tokens = random_tokens(config["vocab"], 11, 3)
    _, after = sorizen_plain.forward(config, weights, tokens)
    replayer = TraceReplayer(folder, "float32", 64, block_len=4, device="cpu")
    seen = []
    for block in replayer.runner.model.blocks:
        original = block.forward

        def spy(streams, pending, ctx, cache, original=original):
            out = original(streams, pending, ctx, cache)
            seen.append(streams.total(out))
            return out

        block.forward = spy
    replayer.run_step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": [0]}], "end": ["a"]})
    assert len(seen) == after.shape[0]
    for run, (got, want) in enumerate(zip(seen, after)):
        assert torch.allclose(got.double(), want, rtol=2e-4, atol=2e-4), f"layer {run}"


def greedy_plain(config, weights, prompt, new):
    tokens = list(prompt)
    for _ in range(new):
        logits, _ = sorizen_plain.forward(config, weights, tokens)
        tokens.append(int(torch.argmax(logits[-1])))
    return tokens[len(prompt):]


def generation(folder, config, weights, dtype, device, lookahead=1, graphs=False):
    from einf_b200.config.engine import EngineConfig
    from einf_b200.engine import Engine

    prompts = [random_tokens(config["vocab"], n, 50 + n) for n in (3, 11, 1, 17, 6, 9)]
    engine = Engine.from_folder(folder, EngineConfig(
        dtype=dtype, block_len=4, num_blocks=64, max_batch_len=16, max_prefill_chunk_len=5, max_requests=4,
        device=device, use_cuda_graphs=graphs, decode_lookahead=lookahead))
    return prompts, engine.generate(prompts, 8)


def test_greedy_generation_through_the_entry_point_emulated(folders, emulated):
    folder, config, weights = folders["mix"]
    prompts, got = generation(folder, config, weights, "float32", "cpu")
    for prompt, tokens in zip(prompts, got):
        assert tokens == greedy_plain(config, weights, prompt, 8)


def test_command_line_runs_the_design(folders, emulated, capsys, tmp_path):
    from einf_b200.cli.run_qwen import main

    folder, config, weights = folders["mix"]
    prompt = [5, 17, 3, 90, 4, 8, 2]
    code = main(["--model-dir", str(folder), "--prompt-ids", ",".join(map(str, prompt)), "--dtype", "float32",
                 "--max-new-len", "5", "--max-prefill-chunk-len", "3", "--block-len", "4", "--max-requests", "2",
                 "--device", "cpu", "--compare-reference"], prog="run_model")
    out = capsys.readouterr().out
    assert code == 0, out
    fields = dict(line.split(": ", 1) for line in out.splitlines() if ": " in line)
    assert json.loads(fields["generated_ids"]) == greedy_plain(config, weights, prompt, 5)
    assert fields["tokens_equal"] == "True" and fields["completion_reason"] == "length"
    # random weights from a bare config.json of the design
    path = tmp_path / "config.json"
    path.write_text(json.dumps(CONFIGS["ones"]))
    code = main(["--random-weights", "--config", str(path), "--seed", "3", "--prompt-ids", "7,8,9", "--dtype", "float32",
                 "--max-new-len", "4", "--block-len", "8", "--device", "cpu"])
    out = capsys.readouterr().out
    assert code == 0 and "generated_ids: [" in out, out


# ---------------------------------------------------------------------------
# keys that decide a row.  The weights are made for it: the first latent dimensions are the first
# dimensions of the normed stream as they are, every head's plain query and key are those (the query
# negated, so that a token is its own worst match), and token 1's embedding is the negative of token
# 0's: token 1 (the needle) is the best match of token 0 (the asker) by far.  The values come from
# other latent dimensions, so they differ.
def needle_model(kind, size, heads=2, scale=2.5, sink=-20.0, rank=24, rot_dim=4):
    config = model(32, 40, [layer(kind, heads, 8, rot_dim, 12, rank, size, None, scale=scale, scaling=yarn(2.0, 32))],
                   streams=2, scale=1.0)
    weights = sorizen_plain.random_model(config, 5)
    width = 32
    down = torch.zeros(rank + rot_dim, width)
    down[:8, :8] = torch.eye(8)                                    # what the scores are made of
    down[8:rank] = weights["l0.mix.dkv"].float()[8:rank] * 0.5
    weights["l0.mix.dkv"] = down.to(torch.bfloat16)                # no rotated key part: the match holds at any distance
    q = torch.zeros(heads, 8 + rot_dim, width)
    q[:, :8, :8] = -torch.eye(8)
    weights["l0.mix.q"] = q.reshape(-1, width).to(torch.bfloat16)
    up = torch.zeros(heads, 8, rank)
    up[:, :, :8] = torch.eye(8)
    weights["l0.mix.uk"] = up.reshape(-1, rank).to(torch.bfloat16)
    weights["l0.mix.dkv.norm"] = torch.ones(rank, dtype=torch.bfloat16)
    weights["l0.norm1"] = torch.ones(width, dtype=torch.bfloat16)
    weights["l0.norm1.b"] = torch.zeros(width, dtype=torch.bfloat16)
    weights["embed"][0, :8] = 3.0 * torch.sign(weights["embed"][0, :8])
    weights["embed"][1] = -weights["embed"][0]
    if kind == SINK:
        weights["l0.mix.sink"] = torch.full((heads,), sink, dtype=torch.bfloat16)
    return config, weights


def needle_tokens(size, needles, length):
    tokens = [2 + (i * 7) % 37 for i in range(length)]
    askers = []
    for n in needles:
        tokens[n] = 1
        tokens[n + size - 1] = 0         # sees the needle at the window's far edge
        tokens[n + size] = 0             # one position on: out of sight
        askers.append((n + size - 1, n + size))
    return tokens, askers


def window_needle_check(tmp_path, kind, dtype, device, size, page, needles, length, rank=24):
    from einf_b200.engine.replay import TraceReplayer

    config, weights = needle_model(kind, size, rank=rank)
    folder = tmp_path / f"needle{size}"
    write_folder(folder, config, 0, weights)
    tokens, askers = needle_tokens(size, needles, length)
    requests = {"n": tokens}
    expected, _ = expected_rows(config, weights, requests)
    # the plain statement itself must feel the edge: one position on, the needle is out of sight
    for inside, outside in askers:
        assert np.abs(expected[("n", inside)] - expected[("n", outside)]).max() > 0.3
    room = -(-length // 64) * 64
    for steps in (trace_tools.whole(requests), trace_tools.last_one_by_one(requests, tail=length - needles[0] - 2),
                  trace_tools.in_portions(requests, sizes=(size - 1, 2, size, 3, 2))):
        replayer = TraceReplayer(folder, dtype, room, block_len=page, device=device)
        check(trace_tools.run_steps(replayer, steps), expected, dtype)


@pytest.mark.parametrize("kind", [SINK, GATE])
def test_a_key_at_the_windows_edge_decides_the_row_emulated(kind, tmp_path, emulated):
    # window 24, pages of 16: the second needle's edge is the page border at 48
    window_needle_check(tmp_path, kind, "float32", "cpu", 24, 16, needles=(0, 25, 60), length=90)


def far_key_check(tmp_path, dtype, device, rank=24):
    """Without a window a key hundreds of positions back still decides a row."""
    from einf_b200.engine.replay import TraceReplayer

    config, weights = needle_model(GATE, None, rank=rank)
    folder = tmp_path / "far"
    write_folder(folder, config, 0, weights)
    length = 330
    tokens = [2 + (i * 7) % 37 for i in range(length)]
    with_needle = list(tokens)
    with_needle[4] = 1
    with_needle[-1] = tokens[-1] = 0
    with_needle[300] = tokens[300] = 0
    requests = {"with": with_needle, "without": tokens}
    expected, _ = expected_rows(config, weights, requests)
    assert np.abs(expected[("with", length - 1)] - expected[("without", length - 1)]).max() > 0.3
    for steps in (trace_tools.whole(requests), trace_tools.last_one_by_one(requests, tail=40),
                  trace_tools.in_portions(requests, sizes=(129, 2, 64, 3))):
        replayer = TraceReplayer(folder, dtype, 704, block_len=16, device=device)
        check(trace_tools.run_steps(replayer, steps), expected, dtype)


def test_a_far_key_counts_emulated(tmp_path, emulated):
    far_key_check(tmp_path, "float32", "cpu")


def sink_check(tmp_path, dtype, device, rank=24):
    """A sink as large as the scores takes a good part of most rows' weight: left out, counted twice or scaled
    like a score, it shows."""
    from einf_b200.engine.replay import TraceReplayer

    config, weights = needle_model(SINK, 9, scale=0.2, sink=3.0, rank=rank)
    _, without = needle_model(SINK, 9, scale=0.2, sink=-40.0, rank=rank)
    folder = tmp_path / "sink"
    write_folder(folder, config, 0, weights)
    requests = {"s": [2 + (i * 5) % 37 for i in range(40)]}
    expected, _ = expected_rows(config, weights, requests)
    other, _ = expected_rows(config, without, requests)
    assert float(np.quantile([np.abs(expected[key] - other[key]).max() for key in expected], 0.25)) > 0.05
    for steps in (trace_tools.whole(requests), trace_tools.last_one_by_one(requests, tail=20),
                  trace_tools.in_portions(requests, sizes=(5, 2, 9))):
        replayer = TraceReplayer(folder, dtype, 64, block_len=16, device=device)
        check(trace_tools.run_steps(replayer, steps), expected, dtype)


def test_a_sink_takes_its_share_emulated(tmp_path, emulated):
    sink_check(tmp_path, "float32", "cpu")


# ---------------------------------------------------------------------------
# the kernels (GPU)
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_each_mechanism_alone(name, dtype, folders):
    folder, config, weights = for_dtype(folders, name, dtype)
    replay_modes(folder, config, weights, 4, dtype, "cuda:0", lengths=(1, 6, 19, 70))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_replay_modes(name, dtype, folders):
    folder, config, weights = for_dtype(folders, name, dtype)
    replay_modes(folder, config, weights, PAGE[name], dtype, "cuda:0", lengths=(1, 5, 9, 23, 37, 50, 131, 300))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,size,page,needles,rank", [
    (SINK, 24, 16, (0, 25, 60), 24), (GATE, 120, 16, (1, 137, 280), 100), (SINK, 120, 16, (1, 137, 280), 200),
    (GATE, 16, 4, (0, 17, 35), 24), (GATE, 24, 16, (0, 25, 60), 300)])
def test_a_key_at_the_windows_edge_decides_the_row(dtype, kind, size, page, needles, rank, tmp_path):
    window_needle_check(tmp_path, kind, dtype, "cuda:0", size, page, needles, needles[-1] + size + 5, rank)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [24, 100, 260])
def test_a_far_key_counts(dtype, rank, tmp_path):
    far_key_check(tmp_path, dtype, "cuda:0", rank)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [24, 100, 260])
def test_a_sink_takes_its_share(dtype, rank, tmp_path):
    sink_check(tmp_path, dtype, "cuda:0", rank)


@pytest.mark.gpu
def test_long_decoding_passes_the_windows(folders):
    """Three hundred tokens one by one after a short prompt: every window passes over decoded tokens many
    times and its pages come back to the pool."""
    from einf_b200.engine.replay import TraceReplayer

    folder, config, weights = folders["mix"]
    requests = make_requests(config, [310], seed=7)
    expected, sure = expected_rows(config, weights, requests)
    replayer = TraceReplayer(folder, "float32", 320, block_len=PAGE["mix"], device="cuda:0")
    rows = trace_tools.run_steps(replayer, trace_tools.last_one_by_one(requests, tail=300))
    check(rows, expected, "float32", sure)


@pytest.mark.gpu
@pytest.mark.parametrize("lookahead,graphs", [(1, False), (1, True), (4, True)])
def test_greedy_generation_through_the_entry_point(lookahead, graphs, folders):
    folder, config, weights = folders["mix"]
    prompts, got = generation(folder, config, weights, "float32", "cuda:0", lookahead, graphs)
    for prompt, tokens in zip(prompts, got):
        assert tokens == greedy_plain(config, weights, prompt, 8)
