"""Pafivik without a GPU: the configuration reader, the plain implementation's own consistency on cases worked
out by hand, and the engine's logic (batching, paging, state slots, the sum over all layers' results, routed
experts) on the plain PyTorch stand-ins of the kernels, against the plain implementation of the design."""
import io
import math
import os

import pytest
import torch

import helpers
import pafivik_models
import plain_pafivik as plain
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
    from chibillm_b200.config import PafivikConfig
    spec = PafivikConfig.from_dict(pafivik_models.with_rank_keys(pafivik_models.get("P1"))).model_spec()
    lin, delta, att = spec.layers
    assert [s.layer for s in spec.run_order] == [0, 1, 2] and [l.depth_average for l in spec.layers] == [1, 2, 3]
    assert all(l.residual_scale == 0.7 and l.layer_scale and l.mixer_out_norm.eps == 1e-5 for l in spec.layers)
    assert (lin.mixer.kind, lin.mixer.head_dim, lin.mixer.value_dim, len(lin.mixer.decay)) == ("linear_attention", 16, 8, 4)
    m = delta.mixer
    assert (m.num_heads, m.num_kv_heads, m.value_dim, m.conv_taps, m.decay_rank, m.gate_rank) == (4, 2, 24, 4, 6, 10)
    assert att.mixer.biases and att.mixer.position.interleaved and att.mixer.position.rotary_dim == 8
    ff = lin.feed_forward
    assert (ff.num_experts, ff.top, ff.scores, ff.weight_on_input, ff.shared_size, ff.shared_output_gate) == (
        5, 2, "sigmoid", True, 16, True)
    assert (delta.feed_forward.activation, delta.feed_forward.biases) == ("xielu", True)
    assert att.feed_forward.shared_size == 0 and not att.feed_forward.shared_output_gate
    assert spec.tie_output_to_embedding and spec.input_adapters[0].constants()["factor"] == 1.5
    bare = PafivikConfig.from_dict(pafivik_models.with_rank_keys(pafivik_models.get("P2"))).model_spec()
    assert bare.layers[0].feed_forward is None and bare.layers[0].feed_forward_out_norm is None
    assert bare.layers[0].mixer.position.kind == "none" and bare.layers[0].mixer.num_kv_heads == 3
    assert bare.layers[1].mixer.conv_taps == 1 and bare.layers[1].residual_scale == 1.0
    assert bare.input_adapters[0].constants()["factor"] == 1.0


def test_ranks_come_from_the_tensors(tmp_path):
    from chibillm_b200.config import load_config
    cfg = pafivik_models.get("P4")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p4"), seed=1)
    _, _, spec = load_config(folder)
    assert [(l.mixer.decay_rank, l.mixer.gate_rank) for l in spec.layers if l.mixer.kind == "channel_delta"] == [(3, 5), (7, 2)]


def test_config_errors_name_the_key():
    from chibillm_b200.config import ConfigError, PafivikConfig

    def read(change):
        cfg = pafivik_models.with_rank_keys(pafivik_models.get("P1"))
        change(cfg)
        return PafivikConfig.from_dict(cfg)

    for change, word in ((lambda c: c.pop("width"), "width"),
                         (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
                         (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
                         (lambda c: c["layers"][1]["mixer"].pop("gate_rank"), "gate_rank"),
                         (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "rot.dims"),
                         (lambda c: c["layers"][0].update(type="mamba"), "type"),
                         (lambda c: c["layers"][0]["mixer"]["decay"].pop(), "decay"),
                         (lambda c: c["layers"][0]["mixer"].update(decay=[0.5, 1.5, 0.5, 0.5]), "decay"),
                         (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
                         (lambda c: c["layers"][1]["mlp"].update(kind="gated"), "kind"),
                         (lambda c: c.update(residual_mult="x"), "residual_mult")):
        with pytest.raises(ConfigError) as e:
            read(change)
        assert word in str(e.value)


# ------------------------------------------------------------------ the plain implementation, by hand
def d64(x):
    return torch.tensor(x, dtype=torch.float64)


def test_plain_rotation_by_hand():
    """Neighbouring features turn together: pair i at position p by p * base^(-2i/dims); the rest pass."""
    x = d64([[[0.0] * 5], [[1.0, 0.0, 0.0, 2.0, 7.0]]])
    y = plain.rotate_interleaved(x, {"base": 16.0, "dims": 4})[1, 0]
    a0, a1 = 1.0, 16.0 ** -0.5
    want = [math.cos(a0), math.sin(a0), -2 * math.sin(a1), 2 * math.cos(a1), 7.0]
    assert torch.allclose(y, d64(want))


def test_plain_recurrences_by_hand():
    # one head, one key channel, one value column; decay 1/2
    o, S = plain.decayed_outer_sums(d64([[[1.0]], [[2.0]]]), d64([[[3.0]], [[1.0]]]), d64([[[5.0]], [[4.0]]]), [0.5])
    assert o.flatten().tolist() == [15.0, 2 * (7.5 + 4.0)] and S.item() == 11.5
    # the delta rule: S1 = b k v; then g decays it, u = b (v - k S'), and the read-out sees the write
    k = d64([[[1.0]], [[1.0]]])
    o, S = plain.gated_delta(2 * k, k, d64([[[4.0]], [[10.0]]]), d64([[0.5], [0.25]]), d64([[[0.9]], [[0.5]]]))
    s2 = 1.0 + 0.25 * (10.0 - 1.0)                  # S1 = 2, decayed to 1
    assert o.flatten().tolist() == [4.0, 2 * s2] and S.item() == s2
    # a decay acts on its own key channel only
    q = d64([[[1.0, 1.0]], [[1.0, 1.0]]])
    kk = d64([[[1.0, 0.0]], [[0.0, 1.0]]])
    o, S = plain.gated_delta(q, kk, d64([[[2.0]], [[3.0]]]), d64([[1.0], [1.0]]), d64([[[1.0, 1.0]], [[0.25, 0.5]]]))
    assert S[0, :, 0].tolist() == [0.5, 3.0] and o[1, 0, 0].item() == 3.5
    g = plain.channel_decay(d64([[[0.0, 100.0]]]), d64([math.log(2.0)]), d64([[0.0, 0.0]]))
    assert torch.allclose(g, d64([[[0.25, math.exp(-200.0)]]]))      # exp(-2 ln 2), exp(-2 * 100)
    y = plain.causal_conv(d64([[1.0], [2.0], [4.0]]), d64([[0.5, 1.0, 2.0]]))
    assert y.flatten().tolist() == [2.0, 5.0, 10.5]
    assert torch.allclose(plain.unit(d64([3.0, 4.0])), d64([0.6, 0.8]), atol=1e-7)


def test_plain_feed_forwards_by_hand():
    z = d64([-1.0, 0.0, 2.0])
    p, q = d64(0.0), d64(0.0)
    ln2 = math.log(2.0)
    want = [(0.5 + ln2) * math.exp(-1.0) - 0.5, 0.0, ln2 * 4 + 1]      # exp(-1) - 1 + 1
    assert torch.allclose(plain.xielu(z, p, q), d64(want))
    # two experts of one feature; scores 1/2 and sigmoid(1): the second is taken, its score multiplies the input
    h = d64([[2.0]])
    w = {"r.router": d64([[0.0], [0.5]])}
    for e in (0, 1):
        w.update({f"r.e{e}.gate": d64([[1.0 + e]]), f"r.e{e}.up": d64([[3.0]]), f"r.e{e}.down": d64([[1.0]])})
    s = 1 / (1 + math.exp(-1.0))
    x = 2.0 * s
    expert = 2 * x / (1 + math.exp(-2 * x)) * 3 * x
    out = plain.moe_ff(h, {"router": {"experts": 2, "top": 1}}, w, "r.")
    assert abs(out.item() - expert) < 1e-12
    w.update({"r.shared.gate": d64([[1.0]]), "r.shared.up": d64([[1.0]]), "r.shared.down": d64([[1.0]]),
              "r.shared.sg": d64([[-0.5]])})
    out = plain.moe_ff(h, {"router": {"experts": 2, "top": 1}, "shared": {"ff": 1}}, w, "r.")
    assert abs(out.item() - expert - (1 - s) * (4 / (1 + math.exp(-2.0)))) < 1e-12


def test_plain_depth_average_by_hand():
    xs = [d64([1.0, 2.0]), d64([10.0, 20.0]), d64([100.0, 0.0])]
    assert plain.depth_average(xs, d64([0.5, 0.0, 2.0])).tolist() == [200.5, 1.0]


# ------------------------------------------------------------------ the engine on the stand-in kernels
@pytest.mark.parametrize("name,page_size,lengths", [("P1", 4, [1, 30, 75]), ("P2", 16, [2, 40, 70]),
                                                    ("P3", 16, [5, 50]), ("P4", 8, [3, 23, 66])])
def test_cutting_and_batching_on_cpu(tmp_path, name, page_size, lengths):
    cfg = pafivik_models.get(name)
    folder = pafivik_models.write_model(cfg, str(tmp_path / name), seed=11)
    reqs = helpers.random_requests(cfg["vocab"], lengths, seed=4)
    ref = pafivik_models.plain_logits(cfg, 11, reqs)
    runner = cpu_runner(folder, page_size, helpers.round64(max(lengths)))
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (helpers.trace_last_decoded(reqs, 12), "decoded"),
                        (helpers.trace_portions(reqs, seed=2), "portions")):
        got = helpers.run_trace(runner, trace)
        helpers.assert_logits_close(got, ref, helpers.TOL["float32"], f"pafivik {name} cpu {what}")
        runner.cache.check_invariants()
        assert not runner.cache.requests
    mixed_reqs = helpers.random_requests(cfg["vocab"], [20, 64, 9, 50, 33, 2], seed=8)
    mixed_ref = pafivik_models.plain_logits(cfg, 11, mixed_reqs)
    pool = 192
    trace = helpers.trace_mixed(mixed_reqs, pool, seed=6, decode_tail=5)
    assert sum(helpers.round64(len(v)) for v in mixed_reqs.values()) > pool       # pages and slots are reused
    runner2 = cpu_runner(folder, page_size, pool)
    got = helpers.run_trace(runner2, trace)
    helpers.assert_logits_close(got, mixed_ref, helpers.TOL["float32"], f"pafivik {name} cpu mixed")
    runner2.cache.check_invariants()
    assert not runner2.cache.requests


def test_token_by_token_from_the_first(tmp_path):
    """Every token alone, from position 0: the convolutions' histories and both recurrences' states start at zero
    in a slot that another request has just left."""
    cfg = pafivik_models.get("P4")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p4"), seed=3)
    reqs = helpers.random_requests(cfg["vocab"], [45, 38], seed=6)
    ref = pafivik_models.plain_logits(cfg, 3, reqs)
    runner = cpu_runner(folder, 4, 64, max_requests=1)
    got = helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 1000))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "pafivik P4 cpu token by token")


def test_cache_plan_and_state(tmp_path):
    cfg = pafivik_models.get("P1")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p1"), seed=2)
    runner = cpu_runner(folder, 4, 128)
    lin, delta, att = runner.storage.views
    assert tuple(lin.arrays["state"].shape[1:]) == (4, 16, 8) and lin.arrays["state"].dtype == torch.float32
    assert tuple(delta.arrays["state"].shape[1:]) == (4, 16, 24) and delta.arrays["state"].dtype == torch.float32
    assert tuple(delta.arrays["history"].shape[1:]) == (3, 2 * 2 * 16 + 4 * 24)
    assert tuple(att.keys.shape[1:]) == (2, 4, 16) and tuple(att.values.shape[1:]) == (2, 4, 16)


def test_a_step_taken_back_leaves_no_trace(tmp_path):
    from chibillm_b200.engine.batch import StepEntry
    cfg = pafivik_models.get("P1")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p1"), seed=5)
    ids = helpers.random_requests(cfg["vocab"], [21], seed=2)["r0"]
    ref = pafivik_models.plain_logits(cfg, 5, {"a": ids})["a"]
    runner = cpu_runner(folder, 4, 64)
    runner.step([StepEntry("a", ids[:9], [])])
    runner.step([StepEntry("a", [7, 7, 7, 7, 7], [4])], provisional=True)
    runner.rollback_step()
    got = runner.step([StepEntry("a", ids[9:], list(range(len(ids) - 9)))])
    helpers.assert_logits_close({"a": got}, {"a": ref[9:]}, helpers.TOL["float32"], "pafivik rollback")


def test_each_options_weight_is_read(tmp_path):
    """Every tensor of a model changes its logits: nothing is loaded and then left out."""
    cfg = pafivik_models.get("P1")
    ids = helpers.random_requests(cfg["vocab"], [24], seed=9)
    w = pafivik_models.random_weights(cfg, 8)
    g = torch.Generator().manual_seed(0)
    runner = cpu_runner(pafivik_models.write_model(cfg, str(tmp_path / "base"), 8, weights=w), 8, 64)
    base = helpers.run_trace(runner, helpers.trace_whole(ids))["r0"]
    model = runner.model
    for name in w:
        if ".mlp.e" in name and not name.startswith("l2.mlp.e"):
            continue
        changed = {k: v.float() for k, v in w.items()}
        changed[name] = changed[name] + 0.5 * torch.randn(changed[name].shape, generator=g) * changed[name].abs().mean()
        model.bind(changed)
        diff = float((helpers.run_trace(runner, helpers.trace_whole(ids))["r0"] - base).abs().max())
        if ".mlp.e" not in name:                       # (an expert may not have been chosen)
            assert diff > 1e-5, name
        want = pafivik_models.plain_logits(cfg, 0, ids, weights=changed)["r0"]
        got = helpers.run_trace(runner, helpers.trace_whole(ids))["r0"]
        assert float((got - want).abs().max()) < 1e-4 * float(want.abs().max()), name


def test_sublayers_that_add_into_a_zeroed_array(tmp_path, monkeypatch):
    """The same model with every part adding its result instead of writing it (what a part without
    ``can_overwrite`` does): the bias of the dense feed-forward then joins through the part itself."""
    from chibillm_b200.parts import attention, channel_delta, linear_attention, mlp
    cfg = pafivik_models.get("P1")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p1"), seed=13)
    reqs = helpers.random_requests(cfg["vocab"], [33], seed=3)
    ref = pafivik_models.plain_logits(cfg, 13, reqs)
    for part in (attention.PagedAttention, channel_delta.ChannelDelta, linear_attention.LinearAttention, mlp.DenseMLP,
                 mlp.RoutedExperts):
        monkeypatch.setattr(part, "can_overwrite", False)
    got = helpers.run_trace(cpu_runner(folder, 4, 64), helpers.trace_portions(reqs, seed=2))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "pafivik, sublayers added")


def test_spec_combinations_that_are_refused():
    from dataclasses import replace
    from chibillm_b200.config import PafivikConfig
    from chibillm_b200.engine.model import DecoderModel
    from chibillm_b200.parts import Runtime
    spec = PafivikConfig.from_dict(pafivik_models.with_rank_keys(pafivik_models.get("P1"))).model_spec()
    rt = Runtime(torch.device("cpu"), torch.float32, ReferenceKernels())
    DecoderModel(spec, rt)

    def with_layer(i, **changes):
        layers = list(spec.layers)
        layers[i] = replace(layers[i], **changes)
        return replace(spec, layers=tuple(layers))

    for bad in (with_layer(1, depth_average=1),                                            # not its place in the order
                with_layer(2, depth_average=None),                                         # some layers, not all
                with_layer(2, mixer=replace(spec.layers[2].mixer, tied_values=True, biases=False)),
                with_layer(1, mixer=replace(spec.layers[1].mixer, num_kv_heads=3)),
                with_layer(0, mixer=replace(spec.layers[0].mixer, decay=(0.5,))),
                with_layer(0, feed_forward=replace(spec.layers[0].feed_forward, gated=False)),
                with_layer(1, feed_forward=replace(spec.layers[1].feed_forward, activation="gelu"))):
        with pytest.raises(ValueError):
            DecoderModel(bad, rt)


def test_random_model_folder_of_the_package(tmp_path):
    """``write_random_model`` takes a Pafivik configuration; the folder runs and agrees with the plain
    implementation on the stored weights."""
    from chibillm_b200.weights import write_random_model
    from safetensors import safe_open
    cfg = pafivik_models.get("P4")
    folder = write_random_model(pafivik_models.with_rank_keys(cfg), str(tmp_path / "random"), seed=2)
    weights = {}
    with safe_open(os.path.join(folder, "model.safetensors"), framework="pt") as f:
        for name in f.keys():
            weights[name] = f.get_tensor(name)
    own = pafivik_models.random_weights(cfg, 0)
    assert {k: tuple(v.shape) for k, v in weights.items()} == {k: tuple(v.shape) for k, v in own.items()}
    reqs = helpers.random_requests(cfg["vocab"], [30], seed=1)
    ref = pafivik_models.plain_logits(cfg, 0, reqs, weights=weights)
    got = helpers.run_trace(cpu_runner(folder, 4, 64), helpers.trace_portions(reqs, seed=1))
    helpers.assert_logits_close(got, ref, helpers.TOL["float32"], "pafivik random folder")


def test_command_line_and_scheduler_on_cpu(tmp_path):
    """Four prompts through the package's command line with room for three at a time and portions of 8
    tokens: every greedy token is the plain implementation's best one (wherever that leads by more than
    rounding)."""
    from chibillm_b200 import cli
    cfg = pafivik_models.get("P1")
    folder = pafivik_models.write_model(cfg, str(tmp_path / "p1"), seed=4)
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
        ref = pafivik_models.plain_logits(cfg, 4, {"a": prompt + new})["a"]
        for i, tok in enumerate(new):
            row = ref[len(prompt) + i - 1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 1e-4 * float(row.abs().max()):
                assert int(torch.argmax(row)) == tok
