"""Lefavik without a GPU: the configuration reader, the plain implementation's own consistency on cases worked
out by hand, and the engine's logic (batching, paging, borrowed caches, windows, learned positions) on the plain
PyTorch stand-ins of the kernels, against the plain implementation of the design."""
import io
import math
import os

import pytest
import torch

import helpers
import lefavik_models
import plain_lefavik as plain
from reference_ops import ReferenceKernels


def cpu_runner(folder, page_size, pool_tokens, max_requests=4):
    from chibillm_b200.engine.runner import ModelRunner
    runner = ModelRunner.from_folder(folder, dtype="float32", device="cpu", page_size=page_size,
                                     pool_tokens=pool_tokens, max_requests=max_requests,
                                     kernels=ReferenceKernels())
    runner.storage.poison()
    return runner


# ------------------------------------------------------------------ configuration
def test_parts_follow_the_file():
    from chibillm_b200.config import LefavikConfig
    spec = LefavikConfig.from_dict(lefavik_models.get("L1")).model_spec()
    src, win, reader, late, last = spec.layers
    assert [s.cache_of for s in spec.run_order] == [None, None, 0, None, 0]
    assert all(l.arrangement == "parallel" and l.feed_forward_norm is None and l.mixer_norm.eps == 1e-5 for l in spec.layers)
    m = src.mixer
    assert (m.num_heads, m.head_dim, m.rope_dim, m.value_dim, m.q_rank, m.kv_rank, m.sink, m.head_gate, m.own_kv) == (
        4, 16, 8, 24, 0, 40, True, True, True)
    assert m.position.interleaved and m.position.theta == 500.0 and m.window is None
    assert not reader.mixer.own_kv and last.mixer.num_heads == 5
    m = win.mixer
    assert (m.num_heads, m.num_kv_heads, m.window, m.query_temperature, m.unit_norm_eps, m.sink_value, m.distance_bias) == (
        6, 3, 5, (0.4, 7), 1e-5, 0.0, "linear")
    assert late.mixer.query_temperature == (-0.1, 50) and late.feed_forward is None
    assert (win.feed_forward.activation, win.feed_forward.intermediate_size) == ("gelu_tanh", 40)
    start = spec.input_adapters[0].constants()
    assert (start["factor"], start["positions"], spec.max_positions) == (2.5, 400, 400)
    assert spec.logit_adapters[0].constants()["factor"] == 0.7 and not spec.tie_output_to_embedding
    bare = LefavikConfig.from_dict(lefavik_models.get("L2")).model_spec()
    m = bare.layers[0].mixer
    assert (m.num_kv_heads, m.value_dim, m.window, m.query_temperature) == (3, 16, None, None)
    assert bare.layers[1].mixer.value_dim == 12 and not bare.logit_adapters
    assert bare.input_adapters[0].constants()["factor"] == 1.0
    masked = LefavikConfig.from_dict(lefavik_models.get("L4")).model_spec()
    assert [l.mixer.cache_window for l in masked.layers if l.mixer.kind == "latent_attention"] == [50, 50]


def test_positions_may_come_from_the_tensor(tmp_path):
    from chibillm_b200.config import load_config
    cfg = lefavik_models.get("L4")
    w = lefavik_models.random_weights(cfg, 1)
    del cfg["max_positions"]
    _, _, spec = load_config(lefavik_models.write_model(cfg, str(tmp_path / "l4"), seed=1, weights=w))
    assert spec.max_positions == 333


def test_config_errors_name_the_key():
    from chibillm_b200.config import ConfigError, LefavikConfig

    def read(change):
        cfg = lefavik_models.get("L1")
        change(cfg["layers"], cfg)
        return LefavikConfig.from_dict(cfg)

    for change, word in ((lambda l, c: c.pop("width"), "width"),
                         (lambda l, c: c.pop("max_positions"), "max_positions"),
                         (lambda l, c: l[0]["mixer"].pop("scale"), "scale"),
                         (lambda l, c: l[0]["mixer"]["rot"].update(dims=6), "rot.dims"),
                         (lambda l, c: l[1]["mixer"].update(kv_heads=4), "kv_heads"),
                         (lambda l, c: l[1]["mixer"]["q_temp"].update(every=0), "every"),
                         (lambda l, c: l[1].update(type="mamba"), "type"),
                         (lambda l, c: l[2]["mixer"].update(kv_from=1), "kv_from"),
                         (lambda l, c: l[2]["mixer"].update(kv_from=2), "kv_from"),
                         (lambda l, c: l[4]["mixer"].update(kv_from=2), "kv_from"),
                         (lambda l, c: l[2]["mixer"].update(kv_rank=41), "kv_rank"),
                         (lambda l, c: l[2]["mixer"]["rot"].update(base=7.0), "rotation"),
                         (lambda l, c: l[0]["mlp"].update(kind="moe"), "kind"),
                         (lambda l, c: c.update(logit_scale="x"), "logit_scale")):
        with pytest.raises(ConfigError) as e:
            read(change)
        assert word in str(e.value)


# ------------------------------------------------------------------ the plain implementation, by hand
def d64(x):
    return torch.tensor(x, dtype=torch.float64)


def test_plain_start_by_hand():
    cfg = {"embedding": {"scale": 2.0}, "norm": {"eps": 0.25}}
    w = {"embed": d64([[0.0, 0.0], [1.0, 2.0]]), "pos": d64([[0.5, -1.0], [1.0, 0.0]]), "embed.norm": d64([1.0, 3.0])}
    x = plain.embed(torch.tensor([1, 1]), cfg, w)
    first, second = [2.5, 3.0], [3.0, 4.0]                     # 2 * (1, 2) + pos
    for row, v in zip(x.tolist(), (first, second)):
        rms = math.sqrt((v[0] ** 2 + v[1] ** 2) / 2 + 0.25)
        assert row == pytest.approx([v[0] / rms, 3 * v[1] / rms])


def test_plain_softmax_by_hand():
    """Two visible keys with scores 0 and ln 3 and a sink of ln 4: weights 1/8 and 3/8; one added (a sink of 0) gives
    1/5 and 3/5; what is not seen gets nothing."""
    s = d64([[0.0, 50.0], [0.0, math.log(3.0)]])
    seen = plain.visible(2)
    assert plain.weights_with_sink(s, seen, d64(math.log(4.0)))[1].tolist() == pytest.approx([1 / 8, 3 / 8])
    w = plain.weights_with_sink(s, seen, d64(0.0))
    assert w[1].tolist() == pytest.approx([1 / 5, 3 / 5]) and w[0].tolist() == pytest.approx([1 / 2, 0.0])
    assert plain.visible(4, 2)[3].tolist() == [False, False, True, True]
    assert plain.visible(3, 1).tolist() == torch.eye(3, dtype=torch.bool).tolist()


def test_plain_temperature_and_slopes_by_hand():
    t = plain.temperature(9, 0.5, 4)
    # positions 0..2: floor((p + 1) / 4) = 0; 3..6: 1; 7..8: 2
    want = [1.0] * 3 + [1 + 0.5 * math.log(2)] * 4 + [1 + 0.5 * math.log(3)] * 2
    assert t.tolist() == pytest.approx(want)
    assert plain.temperature(2, 1.0, 1).tolist() == pytest.approx([1 + math.log(2), 1 + math.log(3)])
    assert plain.slopes(4).tolist() == pytest.approx([2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    assert plain.slopes(3)[0].item() == pytest.approx(2.0 ** (-8 / 3))


def test_plain_rotation_by_hand():
    x = d64([[[0.0] * 4], [[1.0, 0.0, 0.0, 2.0]]])
    y = plain.rotate_neighbours(x, 16.0, 4)[1, 0]
    a0, a1 = 1.0, 16.0 ** -0.5
    assert y.tolist() == pytest.approx([math.cos(a0), math.sin(a0), -2 * math.sin(a1), 2 * math.cos(a1)])


def test_plain_logits_depend_on_the_windows_only():
    """Two plain-attention layers with windows of 5 and 37 positions: a token 40 back cannot be seen through
    both, a token 39 back can; with a latent layer it always can."""
    cfg = lefavik_models.get("L1")
    cfg["layers"] = [cfg["layers"][1], cfg["layers"][3]]
    w = {k: v.double() for k, v in lefavik_models.random_weights(cfg, 5).items()}
    ids = torch.arange(60) % cfg["vocab"]
    base = plain.forward(ids, cfg, w)
    changed = ids.clone()
    changed[10] = 77
    diff = (plain.forward(changed, cfg, w) - base).abs().amax(-1)
    reach = 4 + 36
    assert float(diff[:10].max()) == 0.0 and float(diff[10 + reach]) > 0.0 and float(diff[10 + reach + 1:].max()) == 0.0


# ------------------------------------------------------------------ the engine on the stand-in kernels
@pytest.mark.parametrize("name,page_size,lengths", [("L1", 4, [1, 30, 75]), ("L2", 16, [2, 40, 70]),
                                                    ("L3", 16, [5, 120]), ("L4", 8, [3, 23, 66])])
def test_cutting_and_batching_on_cpu(tmp_path, name, page_size, lengths):
    cfg = lefavik_models.get(name)
    folder = lefavik_models.write_model(cfg, str(tmp_path / name), seed=11)
    reqs = helpers.random_requests(cfg["vocab"], lengths, seed=4)
    ref = lefavik_models.plain_logits(cfg, 11, reqs)
    runner = cpu_runner(folder, page_size, helpers.round64(max(lengths)))
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (helpers.trace_last_decoded(reqs, 12), "decoded"),
                        (helpers.trace_portions(reqs, seed=2), "portions")):
        got = helpers.run_trace(runner, trace)
        helpers.assert_logits_close(got, ref, helpers.TOL["float32"], f"lefavik {name} cpu {what}")
        runner.cache.check_invariants()
        assert not runner.cache.requests
    mixed_reqs = helpers.random_requests(cfg["vocab"], [20, 64, 9, 50, 33, 2], seed=8)
    mixed_ref = lefavik_models.plain_logits(cfg, 11, mixed_reqs)
    pool = 192
    trace = helpers.trace_mixed(mixed_reqs, pool, seed=6, decode_tail=5)
    assert sum(helpers.round64(len(v)) for v in mixed_reqs.values()) > pool       # pages and slots are reused
    runner2 = cpu_runner(folder, page_size, pool)
    got = helpers.run_trace(runner2, trace)
    helpers.assert_logits_close(got, mixed_ref, helpers.TOL["float32"], f"lefavik {name} cpu mixed")
    runner2.cache.check_invariants()
    assert not runner2.cache.requests


def test_token_by_token_from_the_first(tmp_path):
    cfg = lefavik_models.get("L4")
    folder = lefavik_models.write_model(cfg, str(tmp_path / "l4"), seed=3)
    reqs = helpers.random_requests(cfg["vocab"], [60, 38], seed=6)
    ref = lefavik_models.plain_logits(cfg, 3, reqs)
    got = helpers.run_trace(cpu_runner(folder, 4, 64, max_requests=1), helpers.trace_last_decoded(reqs, 1000))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "lefavik L4 cpu token by token")


def test_cache_plan(tmp_path):
    """Readers hold no arrays of their own; a latent row is one array; windows give their pages back, a latent
    layer without one keeps everything."""
    from chibillm_b200.engine.batch import StepEntry
    cfg = lefavik_models.get("L1")
    runner = cpu_runner(lefavik_models.write_model(cfg, str(tmp_path / "l1"), seed=2), 4, 128)
    src, win, reader, late, last = runner.storage.views
    assert tuple(src.keys.shape[1:]) == (1, 4, 48) and src.keys.data_ptr() == src.values.data_ptr() and src.writes
    for r in (reader, last):
        assert r.keys.data_ptr() == src.keys.data_ptr() and not r.writes
    assert tuple(win.keys.shape[1:]) == (3, 4, 16) and tuple(late.values.shape[1:]) == (2, 4, 24)
    ids = helpers.random_requests(cfg["vocab"], [80], seed=1)["r0"]
    runner.step([StepEntry("a", ids, [])])
    held = {g.window: g.num_pages - runner.cache.free_pages(g.name) for g in runner.plan.groups}
    assert held[None] == 20 and held[5] <= 3 and held[37] <= 11


def test_no_position_beyond_the_table(tmp_path):
    from chibillm_b200.engine.batch import BatchError, StepEntry
    cfg = lefavik_models.get("L2")
    cfg["max_positions"] = 20
    folder = lefavik_models.write_model(cfg, str(tmp_path / "l2"), seed=2)
    runner = cpu_runner(folder, 4, 64)
    ids = helpers.random_requests(cfg["vocab"], [21], seed=1)["r0"]
    ref = lefavik_models.plain_logits(cfg, 2, {"a": ids[:20]})["a"]
    got = runner.step([StepEntry("a", ids[:20], [19])])
    helpers.assert_logits_close({"a": got}, {"a": ref[19:]}, helpers.TOL["float32"], "lefavik last position")
    with pytest.raises(BatchError):
        runner.step([StepEntry("a", ids[20:], [0])])


def test_each_tensor_is_read(tmp_path):
    """Every tensor of a model changes its logits as the plain implementation says: nothing is loaded and left out."""
    cfg = lefavik_models.get("L1")
    ids = helpers.random_requests(cfg["vocab"], [48], seed=9)
    w = lefavik_models.random_weights(cfg, 8)
    g = torch.Generator().manual_seed(0)
    runner = cpu_runner(lefavik_models.write_model(cfg, str(tmp_path / "base"), 8, weights=w), 8, 64)
    base = helpers.run_trace(runner, helpers.trace_whole(ids))["r0"]
    for name in w:
        changed = {k: v.float() for k, v in w.items()}
        changed[name] = changed[name] + 0.5 * torch.randn(changed[name].shape, generator=g) * changed[name].abs().mean()
        runner.model.bind(changed)
        got = helpers.run_trace(runner, helpers.trace_whole(ids))["r0"]
        assert float((got - base).abs().max()) > 1e-5, name
        want = lefavik_models.plain_logits(cfg, 0, ids, weights=changed)["r0"]
        assert float((got - want).abs().max()) < 1e-4 * float(want.abs().max()), name


def test_branches_through_an_array_of_their_own(tmp_path, monkeypatch):
    """The same model with the parallel block's other ways: parts that cannot leave their last product to the
    block, and the branches summed in an array of their own before they join the residual."""
    from chibillm_b200.parts import attention, block, latent_attention, mlp
    cfg = lefavik_models.get("L1")
    folder = lefavik_models.write_model(cfg, str(tmp_path / "l1"), seed=13)
    reqs = helpers.random_requests(cfg["vocab"], [33], seed=3)
    ref = lefavik_models.plain_logits(cfg, 13, reqs)
    for part in (attention.PagedAttention, latent_attention.LatentAttention, mlp.GatedMLP):
        monkeypatch.setattr(part, "can_hold", False)
    got = helpers.run_trace(cpu_runner(folder, 4, 64), helpers.trace_portions(reqs, seed=2))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "lefavik, one branch after the other")
    runner = cpu_runner(folder, 4, 64)
    for b in runner.model.blocks:
        b.direct = b.hold = b.scaled_ok = False
    got = helpers.run_trace(runner, helpers.trace_portions(reqs, seed=2))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "lefavik, branches apart")


def test_spec_combinations_that_are_refused():
    from dataclasses import replace
    from chibillm_b200.config import LefavikConfig
    from chibillm_b200.engine.model import DecoderModel
    from chibillm_b200.parts import Runtime
    spec = LefavikConfig.from_dict(lefavik_models.get("L1")).model_spec()
    rt = Runtime(torch.device("cpu"), torch.float32, ReferenceKernels())
    DecoderModel(spec, rt)

    def with_mixer(i, **changes):
        layers = list(spec.layers)
        layers[i] = replace(layers[i], mixer=replace(layers[i].mixer, **changes))
        return replace(spec, layers=tuple(layers))

    for bad in (with_mixer(1, sink=True), with_mixer(1, biases=True), with_mixer(1, softcap=10.0),
                with_mixer(1, output_gate=True), with_mixer(0, q_rank=16), with_mixer(0, rope_dim=7)):
        with pytest.raises(ValueError):
            DecoderModel(bad, rt)


def test_random_model_folder_of_the_package(tmp_path):
    """``write_random_model`` takes a Lefavik configuration; the folder runs and agrees with the plain
    implementation on the stored weights."""
    from chibillm_b200.weights import write_random_model
    from safetensors import safe_open
    cfg = lefavik_models.get("L4")
    folder = write_random_model(cfg, str(tmp_path / "random"), seed=2)
    weights = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name)
    own = lefavik_models.random_weights(cfg, 0)
    assert {k: tuple(v.shape) for k, v in weights.items()} == {k: tuple(v.shape) for k, v in own.items()}
    reqs = helpers.random_requests(cfg["vocab"], [30], seed=1)
    ref = lefavik_models.plain_logits(cfg, 0, reqs, weights=weights)
    got = helpers.run_trace(cpu_runner(folder, 4, 64), helpers.trace_portions(reqs, seed=1))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "lefavik random folder")


def test_command_line_and_scheduler_on_cpu(tmp_path):
    """Four prompts through the package's command line with room for three at a time and portions of 8
    tokens: every greedy token is the plain implementation's best one (wherever that leads by more than
    rounding)."""
    from chibillm_b200 import cli
    cfg = lefavik_models.get("L1")
    folder = lefavik_models.write_model(cfg, str(tmp_path / "l1"), seed=4)
    prompts = list(helpers.random_requests(cfg["vocab"], [1, 7, 23, 30], seed=1).values())
    argv = ["--context-length", "64", "--max-tokens", "5", "--max-seqs", "3", "--max-batch-tokens", "16",
            "--prefill-chunk", "8", "--dtype", "float32", "--ignore-eos", "--no-stream"]
    for p in prompts:
        argv += ["--prompt-ids", ",".join(map(str, p))]
    out, err = io.StringIO(), io.StringIO()
    assert cli.run(cli.parse_cli_options(argv + [folder]), io.StringIO(""), out, err,
                   kernels=ReferenceKernels(), device="cpu") == 0, err.getvalue()
    replies = [[int(t) for t in line.split()] for line in out.getvalue().splitlines()]
    assert len(replies) == 4 and all(len(r) == 5 for r in replies)
    for prompt, new in zip(prompts, replies):
        ref = lefavik_models.plain_logits(cfg, 4, {"a": prompt + new})["a"]
        for i, tok in enumerate(new):
            row = ref[len(prompt) + i - 1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 1e-4 * float(row.abs().max()):
                assert int(torch.argmax(row)) == tok
