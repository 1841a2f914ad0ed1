"""Pafivik on the GPU against the plain implementation of the design (tests/plain_pafivik.py): each mechanism's
kernels alone -- the two recurrences in portions of all lengths (chunks, borders of chunks, single tokens) from
used slots, a value that survives long, strong decays; the convolution; attention with biases and a rotation
of neighbouring features, one key made to stand out; the norm before a gate; xIELU; the sigmoid router; experts
with weighted inputs beside a gated shared one; a sublayer's end with the sum over all results -- then one
layer of each kind alone and whole models through the step function: whole prompts, the last tokens one by
one, portions down to two tokens, mixed batches with reused pages and slots, long decoding; then greedy
generation through the package's entry point and the trace program."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import helpers
import pafivik_models
import plain_pafivik as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KTOL = {"float32": 2e-5, "bfloat16": 2e-2}


@pytest.fixture(scope="module")
def kernels():
    from chibillm_b200.kernels.ops import CudaKernels
    return CudaKernels(torch.device(DEV))


def close(got, ref, tol, what):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: not finite"
    worst = float((got - ref).abs().max())
    scale = float(ref.abs().max())
    assert worst <= tol * max(scale, 1e-30), f"{what}: max |diff| {worst:.3e} > {tol:.1e} * {scale:.3e}"


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def rounded(t, dtype):
    return t.to(DTYPES[dtype]).double()


# ------------------------------------------------------------------ the recurrences
def run_in_steps(lens, steps, state, slots, rows, outs_width, call):
    """Feeds sequences side by side: a step gives every sequence its next tokens (0: left out).  ``call`` gets the
    step's rows of each array in ``rows``, o, q_start, slots and the longest portion."""
    pos, got = [0] * len(lens), [[] for _ in lens]
    for step in steps:
        ns = [min(n, lens[s] - pos[s]) for s, n in enumerate(step)]
        live = [s for s in range(len(lens)) if ns[s] > 0]
        if not live:
            continue
        args = [torch.cat([r[s][pos[s]:pos[s] + ns[s]] for s in live]).to(DEV) for r in rows]
        o = torch.full((args[0].shape[0], outs_width), float("nan"), dtype=torch.float32, device=DEV)
        call(args, o, i32([0] + list(np.cumsum([ns[s] for s in live]))), i32([slots[s] for s in live]), max(ns))
        at = 0
        for s in live:
            got[s].append(o[at:at + ns[s]].cpu())
            at += ns[s]
            pos[s] += ns[s]
    assert pos == list(lens)
    return [torch.cat(g) for g in got]


# portions: whole; chunk borders, just before and after; two tokens; single ones; one sequence left out at times
CUTS = {"whole": [(1000, 1000, 1000)],
        "borders": [(16, 15, 1), (1, 17, 0), (15, 2, 33), (17, 1, 16), (1000, 1000, 1000)],
        "small": [(5, 3, 2), (2, 2, 0), (1, 0, 7), (4, 6, 1), (33, 31, 1), (1, 1, 1), (1000, 1000, 1000)],
        "tokens": [(2, 1, 1)] + [(1, 1, 1)] * 90}
DELTA_SHAPES = [(4, 2, 16, 8), (3, 3, 10, 7), (2, 2, 64, 64), (6, 2, 12, 33), (2, 1, 128, 128), (4, 4, 100, 40),
                (1, 1, 130, 20), (2, 2, 256, 16), (1, 1, 300, 9), (16, 8, 64, 48), (40, 40, 64, 64), (12, 12, 128, 136)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,e", DELTA_SHAPES)
def test_gated_delta_rule(kernels, dtype, H, G, d, e):
    """Three sequences side by side in slots that others have used, in all ways of cutting, against the plain
    recurrence over the whole sequences; the kept states are compared too.  Some heads hardly decay, some
    forget within a token, some keys repeat (the writes then correct one another)."""
    g = torch.Generator().manual_seed(H * 1000 + d)
    dt = DTYPES[dtype]
    lens = [90, 61, 53]
    big = H * d * e > 100000
    qkv, logits, beta = [], [], []
    for n in lens:
        x = torch.randn(n, 2 * G * d + H * e, generator=g)
        x[n // 2:n // 2 + 3, G * d:2 * G * d] = x[0, G * d:2 * G * d]              # the first key once more, three times
        qkv.append(x.to(dt))
        logits.append(torch.randn(n, H * d, generator=g) * 2)
        beta.append((torch.randn(n, H, generator=g) * 2).to(dt))
    a_log = torch.linspace(-6.0, 3.0, H) if H > 1 else torch.zeros(1)
    dt_bias = torch.rand(H * d, generator=g) * 4 - 3
    refs, states = [], []
    for x, z, b in zip(qkv, logits, beta):
        n = x.shape[0]
        x = x.double()
        q = plain.unit(x[:, :G * d].view(n, G, d)).repeat_interleave(H // G, 1) * d ** -0.5
        k = plain.unit(x[:, G * d:2 * G * d].view(n, G, d)).repeat_interleave(H // G, 1)
        decay = plain.channel_decay(z.double().view(n, H, d), a_log.double(), dt_bias.double().view(H, d))
        v, sb = x[:, 2 * G * d:].view(n, H, e), torch.sigmoid(b.double())
        S = torch.zeros(H, d, e, dtype=torch.float64)
        o = torch.zeros(n, H, e, dtype=torch.float64)
        for t in range(n):                              # (plain.gated_delta, all heads at once)
            S = decay[t][:, :, None] * S
            u = sb[t][:, None] * (v[t] - torch.einsum("hde,hd->he", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            o[t] = torch.einsum("hde,hd->he", S, q[t])
        if not big:
            o2, S2 = plain.gated_delta(q[:6], k[:6], v[:6], sb[:6], decay[:6])
            assert torch.allclose(o2, o[:6])
        refs.append(o.reshape(n, H * e))
        states.append(S)
    tol = 2e-5                                          # (the inputs are given in the kernel's own type)
    if dtype == "bfloat16":
        tol = 1e-4
    for name in (("whole", "borders", "small") if big else CUTS):
        state = torch.full((5, H, d, e), 7.0, device=DEV)
        slots = [3, 0, 4]
        state[slots] = 0.0                              # what admission does to a slot

        def call(args, o, q_start, sl, longest):
            kernels.channel_delta(args[0], args[1], args[2], a_log.to(DEV), dt_bias.to(DEV), state, o, q_start, sl, H, G, d, e,
                                  1e-6, d ** -0.5, longest)

        got = run_in_steps(lens, CUTS[name], state, slots, (qkv, logits, beta), H * e, call)
        for s in range(3):
            close(got[s], refs[s], tol, f"delta rule {H} {G} {d} {e} {dtype} {name} sequence {s}")
            close(state[slots[s]], states[s], tol, f"delta rule's state {H} {G} {d} {e} {dtype} {name} sequence {s}")
        assert float((state[[1, 2]] - 7.0).abs().max()) == 0.0       # slots of nobody are not touched


LINEAR_SHAPES = [(4, 16, 8), (3, 9, 14), (2, 64, 64), (5, 12, 33), (2, 128, 128), (3, 100, 40), (1, 130, 20), (2, 256, 16),
                 (1, 300, 9), (40, 64, 64), (12, 128, 136)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("activate", [True, False])
@pytest.mark.parametrize("H,d,e", LINEAR_SHAPES)
def test_linear_attention_with_constant_decays(kernels, dtype, H, d, e, activate):
    g = torch.Generator().manual_seed(H * 1000 + d + e)
    dt = DTYPES[dtype]
    lens = [90, 61, 53]
    big = H * d * e > 100000
    wide = [torch.randn(n, H * (2 * d + e) + 8, generator=g).to(dt) for n in lens]       # columns of a wider array
    decay = torch.tensor([1.0, 0.0, 0.999, 0.3] * H)[:H]
    refs, states = [], []
    for x in wide:
        n = x.shape[0]
        x = x[:, :H * (2 * d + e)].double()
        x = plain.silu(x) if activate else x
        q, k, v = x[:, :H * d].view(n, H, d), x[:, H * d:2 * H * d].view(n, H, d), x[:, 2 * H * d:].view(n, H, e)
        S = torch.zeros(H, d, e, dtype=torch.float64)
        o = torch.zeros(n, H, e, dtype=torch.float64)
        for t in range(n):
            S = decay.double()[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
            o[t] = torch.einsum("hde,hd->he", S, q[t])
        if not big:
            assert torch.allclose(plain.decayed_outer_sums(q[:6], k[:6], v[:6], decay.double())[0], o[:6])
        refs.append(o.reshape(n, H * e))
        states.append(S)
    tol = 2e-5 if dtype == "float32" or not activate else 1e-4
    for name in (("whole", "borders", "small") if big else CUTS):
        state = torch.full((5, H, d, e), 7.0, device=DEV)
        slots = [3, 0, 4]
        state[slots] = 0.0

        def call(args, o, q_start, sl, longest):
            kernels.decayed_attention(args[0][:, :H * (2 * d + e)], decay.to(DEV), state, o, q_start, sl, H, d, e, longest,
                                      activate=activate)

        got = run_in_steps(lens, CUTS[name], state, slots, (wide,), H * e, call)
        for s in range(3):
            close(got[s], refs[s], tol, f"linear attention {H} {d} {e} {dtype} {name} sequence {s}")
            close(state[slots[s]], states[s], tol, f"linear attention's state {H} {d} {e} {dtype} {name} sequence {s}")
        assert float((state[[1, 2]] - 7.0).abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("portions", [[700], [7, 300, 1, 1, 391], [300] + [1] * 400])
def test_what_the_first_token_wrote_is_there_700_tokens_later(kernels, dtype, portions):
    """One head hardly decays and nobody writes at the first token's key again: the last token's query finds
    the first value, times the product of the decays.  The other head forgets it at once.  A read-out
    before the write, a decay on the wrong rows or a lost state would show as zero."""
    H, d, e, T = 2, 32, 8, 700
    dt = DTYPES[dtype]
    x = torch.zeros(T, 2 * H * d + H * e)
    q, k, v = x[:, :H * d].view(T, H, d), x[:, H * d:2 * H * d].view(T, H, d), x[:, 2 * H * d:].view(T, H, e)
    k[0, :, 5] = 1.0
    k[1:, :, 6] = 1.0                                    # everybody else writes elsewhere
    q[:, :, 5] = 2.0                                     # (made a unit vector: 1)
    v[0] = 3.0
    v[1:] = -9.0
    z = torch.full((T, H * d), -12.0)                    # softplus: 6.1e-6
    z[:, d:] = 6.0
    beta = torch.full((T, H), 30.0).to(dt)               # sigmoid: 1
    state = torch.zeros(1, H, d, e, device=DEV)
    got, pos = [], 0
    for n in portions:
        o = torch.empty(n, H * e, device=DEV)
        kernels.channel_delta(x[pos:pos + n].to(dt).to(DEV), z[pos:pos + n].to(DEV), beta[pos:pos + n].to(DEV),
                              torch.zeros(H, device=DEV), torch.zeros(H * d, device=DEV), state, o, i32([0, n]), i32([0]), H, H,
                              d, e, 1e-6, d ** -0.5, n)
        got.append(o.cpu())
        pos += n
    got = torch.cat(got).view(T, H, e)
    want0 = 3.0 * d ** -0.5
    assert float((got[0] - want0).abs().max()) < 1e-4    # the first token's own read-out sees its write
    step = math.log1p(math.exp(-12.0))
    tol = 1e-5 if dtype == "float32" else 1e-3
    for t in (1, 15, 16, 17, 307, 308, 309, T - 1):
        assert abs(float(got[t, 0, 0]) / (want0 * math.exp(-step * t)) - 1) < tol, t
        forgotten = want0 * math.exp(-math.log1p(math.exp(6.0)) * t)
        assert abs(float(got[t, 1, 0]) - forgotten) <= 1e-3 * forgotten + 1e-30


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,taps", [(40, 1), (40, 2), (64, 3), (128, 4), (24, 5), (7, 3), (4096, 3)])
def test_convolution_over_portions(kernels, dtype, C, taps):
    """Portions shorter than the taps, single tokens, a slot that another request has used; without a bias."""
    g = torch.Generator().manual_seed(C + taps)
    dt = DTYPES[dtype]
    lens = [70, 29, 41]
    xs = [torch.randn(n, C + 8, generator=g).to(dt) for n in lens]
    w = torch.randn(C, taps, generator=g)
    history = torch.full((4, max(taps - 1, 1), C), 9.0, dtype=dt, device=DEV)
    slots = [3, 0, 2]
    history[slots] = 0.0
    outs = []

    def call(args, o, q_start, sl, longest):
        out = torch.empty(args[0].shape[0], C, dtype=dt, device=DEV)
        kernels.causal_conv(args[0][:, :C], w.to(DEV), None, history, out, q_start, sl, longest, activation="silu",
                            weight_t=w.t().contiguous().to(DEV))
        o.copy_(out.float())

    for cut in ([(1000,) * 3], [(1, 2, 3), (2, 1, 0), (1, 1, 1), (3, 0, 2), (9, 8, 17), (1, 1, 1), (1000,) * 3]):
        history[slots] = 0.0
        outs = run_in_steps(lens, cut, None, slots, (xs,), C, call)
        for s in range(3):
            close(outs[s], plain.silu(plain.causal_conv(xs[s][:, :C].double(), w.double())), KTOL[dtype],
                  f"convolution {C} {taps} {dtype} sequence {s}")
            if taps > 1:
                close(history[slots[s]], xs[s][lens[s] - taps + 1:, :C], 1e-30, "kept inputs")
    assert float((history[1].float() - 9.0).abs().max()) == 0.0


# ------------------------------------------------------------------ attention
def run_attention(kernels, q, k, v, bias, rot, dtype, page_size, portions, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e] of one sequence through the kernel that adds the biases, rotates
    and appends, and the attention kernel, with pages given out in a scrambled order; the rows of q and k in
    the order in which the part binds them.  Returns [T, H, e]."""
    from chibillm_b200.config.spec import PositionSpec
    from chibillm_b200.parts import Runtime, make_position
    dt = DTYPES[dtype]
    T, H, d = q.shape
    G, e = k.shape[1], v.shape[2]
    inv_freq, dims, order = None, 0, torch.arange(d)
    if rot:
        position = make_position(PositionSpec(kind="rope", head_dim=d, rotary_dim=rot["dims"], theta=rot["base"],
                                              interleaved=True), Runtime(torch.device(DEV), dt, kernels))
        (inv_freq, dims), order = position.fused_rotation(), position.feature_order()
    pages = (T + page_size - 1) // page_size + 3
    given = torch.randperm(pages, generator=torch.Generator().manual_seed(T))[:pages - 3]
    table = torch.full((2, pages), -1, dtype=torch.int32)
    table[1, :given.numel()] = given.to(torch.int32)
    table = table.to(DEV)
    kc = torch.full((pages, G, page_size, d), float("nan"), dtype=dt, device=DEV)
    vc = torch.full((pages, G, page_size, e), float("nan"), dtype=dt, device=DEV)
    row = torch.cat([q[:, :, order].reshape(T, -1), k[:, :, order].reshape(T, -1), v.reshape(T, -1)], 1).to(dt).to(DEV)
    bq, bk, bv = bias[:H * d].view(H, d), bias[H * d:H * d + G * d].view(G, d), bias[H * d + G * d:]
    b = torch.cat([bq[:, order].reshape(-1), bk[:, order].reshape(-1), bv]).contiguous().to(DEV)
    outs, pos = [], 0
    for n in portions:
        n = min(n, T - pos)
        if n <= 0:
            break
        positions, seq_of, rows = i32(list(range(pos, pos + n))), i32([0] * n), i32([1])
        q_out = torch.empty(n, H * d, dtype=dt, device=DEV)
        kernels.qkv_bias_norm_append(row[pos:pos + n], q_out, kc, vc, b, None, None, None, inv_freq, dims, positions, seq_of,
                                     table, H, G, d, e, page_size, rows)
        out = torch.empty(n, H * e, dtype=dt, device=DEV)
        kernels.attention(q_out, kc, vc, out, table, i32([0, n]), i32([pos + n]), seq_of, positions, H, G, d, page_size,
                          scale, None, n, pos + n, n, rows, value_dim=e)
        outs.append(out.float().cpu().view(n, H, e))
        pos += n
    kernels.check_error_word()
    return torch.cat(outs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,e,rot", [(4, 2, 16, 16, 8), (6, 3, 12, 20, 6), (4, 1, 64, 64, 64), (2, 1, 20, 4, 20),
                                         (8, 2, 32, 48, 16), (3, 3, 128, 128, 128), (2, 2, 10, 10, 0)])
def test_attention_with_biases_and_neighbours_rotated(kernels, dtype, H, G, d, e, rot):
    g = torch.Generator().manual_seed(d * 7 + e)
    T = 150
    q, k, v = torch.randn(T, H, d, generator=g), torch.randn(T, G, d, generator=g), torch.randn(T, G, e, generator=g)
    bias = torch.randn(H * d + G * d + G * e, generator=g) * 0.3
    rotation = {"base": 300.0, "dims": rot} if rot else None
    bq, bk, bv = bias[:H * d].view(H, d), bias[H * d:H * d + G * d].view(G, d), bias[H * d + G * d:].view(G, e)
    qd = plain.rotate_interleaved(rounded(q, dtype) + bq.double(), rotation)
    kd = plain.rotate_interleaved(rounded(k, dtype) + bk.double(), rotation)
    vd = rounded(v, dtype) + bv.double()
    if dtype == "bfloat16":
        qd, kd, vd = rounded(qd, dtype), rounded(kd, dtype), rounded(vd, dtype)
    scale = 1.3 / math.sqrt(d)
    ref = plain.causal_attention(qd, kd, vd, scale)
    for portions in ([T], [40, 2, 1, 1, 70, 3, 33], [100] + [1] * 50):
        got = run_attention(kernels, q, k, v, bias, rotation, dtype, 16, portions, scale)
        close(got, ref, KTOL[dtype], f"attention {H} {G} {d} {e} {rot} {dtype} {portions[:2]}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("e", [16, 24])
def test_one_key_among_hundreds(kernels, dtype, e):
    """One key is made to stand out (its score beats all others by far, its value is known): every later query
    returns its value, no earlier one does.  It sits at the start, at page borders and far back, for rows of a
    prompt and for tokens decoded alone."""
    H, G, d, T, page = 4, 2, 16, 400, 16
    for key_pos in (0, 15, 16, 207, 299, 300):
        g = torch.Generator().manual_seed(key_pos)
        q, k = torch.randn(T, H, d, generator=g) * 0.1 + 1.0, torch.randn(T, G, d, generator=g) * 0.1
        v = torch.randn(T, G, e, generator=g) * 0.01
        k[key_pos] = 3.0
        v[key_pos] = 7.0
        for portions in ([T], [300] + [1] * 100, [3, 2, 290, 2, 1, 1, 1, 2, 98]):
            got = run_attention(kernels, q, k, v, torch.zeros(H * d + G * d + G * e), None, dtype, page, portions, 1.0)
            assert float((got[key_pos:] - 7.0).abs().max()) < 0.1 and (key_pos == 0 or float(got[:key_pos].abs().max()) < 0.1)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_rotation_turns_neighbours(kernels, dtype):
    """A query and a key whose features are equal apart from one neighbouring pair: the score falls with the
    cosine of that pair's angle times the distance, so the softmax over two keys shows which features turn and
    how fast."""
    d, T = 8, 33
    rotation = {"base": 100.0, "dims": 6}
    for pair in range(4):
        q, k = torch.zeros(T, 1, d), torch.zeros(T, 1, d)
        q[:, 0, 2 * pair], k[0, 0, 2 * pair] = 4.0, 4.0                      # the other keys are zero: their scores are 0
        v = torch.zeros(T, 1, 4)
        v[0] = 1.0
        got = run_attention(kernels, q, k, v, torch.zeros(2 * d + 4), rotation, dtype, 4, [20] + [1] * 13, 0.25)
        angle = 100.0 ** (-2.0 * pair / 6) if pair < 3 else 0.0
        for p in range(1, T):
            weight = math.exp(4.0 * math.cos(angle * p))
            assert abs(float(got[p, 0, 0]) - weight / (weight + p)) < (1e-5 if dtype == "float32" else 2e-2), (pair, p)


# ------------------------------------------------------------------ row-wise kernels
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W", [(1, 48), (37, 30), (300, 256), (5, 1000), (3, 5000), (2, 4096), (65, 8192)])
def test_norm_then_gate(kernels, dtype, T, W):
    g = torch.Generator().manual_seed(T + W)
    x, z, w = torch.randn(T, W, generator=g) * 3, torch.randn(T, W, generator=g), 0.5 + torch.rand(W, generator=g)
    ref = plain.rms_norm(x.double(), w.double(), 1e-5) * torch.sigmoid(rounded(z, dtype))
    wide = torch.randn(T, W + 24, generator=g).to(DTYPES[dtype]).to(DEV)      # the gate as a slice of a wider array
    wide[:, 8:8 + W] = z.to(DTYPES[dtype]).to(DEV)
    out = torch.empty(T, W, dtype=DTYPES[dtype], device=DEV)
    kernels.norm_then_gate(x.to(DEV), wide[:, 8:8 + W], w.to(DEV), 1e-5, out)
    close(out, ref, KTOL[dtype], f"norm and gate {T} {W} {dtype}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n", [70, 72, 1024, 68])
@pytest.mark.parametrize("splits", [1, 3])
def test_xielu(kernels, dtype, n, splits):
    """With and without a bias, in place and from a product's partial sums; arguments of all sizes, next to zero
    too, where exp(z) - 1 - z would cancel."""
    from chibillm_b200.kernels.ops import PendingSum
    g = torch.Generator().manual_seed(n)
    T = 33
    z = torch.randn(T, n, generator=g) * torch.logspace(-5, 1.2, n)[None, :]
    bias = torch.randn(n, generator=g) * torch.logspace(-6, 0, n)
    p, q = torch.tensor(0.4), torch.tensor(-1.3)
    pos, neg = float(plain.softplus(p)), 0.5 + float(plain.softplus(q))
    for b in (bias, None):
        out = torch.empty(T, n, dtype=DTYPES[dtype], device=DEV)
        bd = None if b is None else b.to(DEV)
        if splits > 1:
            parts = torch.randn(splits, T, n, generator=g)
            total = parts.double().sum(0)
            kernels.bias_xielu(PendingSum(kernels, parts.to(DEV), splits, T, n), bd, out, pos, neg)
        else:
            total = rounded(z, dtype)
            out.copy_(z)
            kernels.bias_xielu(out, bd, out, pos, neg)
        arg = total + (0 if b is None else b.double())
        ref = plain.xielu(arg, p.double(), q.double())
        err = (out.double().cpu() - ref).abs()
        # of every value by itself, small ones too (but not where the two terms of a negative z cancel)
        bound = (1e-6 if dtype == "float32" else 5e-3) * (ref.abs() + arg.abs())
        if splits > 1:
            bound = bound + 1e-6                        # (of the sum over the splits in 32-bit)
        assert bool((err <= bound + 1e-12).all()), (dtype, n, splits, float((err / bound).max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,n", [(1, 64), (37, 257), (8, 128), (8, 1024), (300, 1024), (3, 4096), (70, 4096), (130, 640),
                                 (5, 12288), (66, 12288), (100, 72)])
@pytest.mark.parametrize("splits", [1, 5, 19])
def test_sublayer_end(kernels, dtype, T, n, splits):
    """residual += vec * y / rms(y) with y a product's partial sums plus a bias, then this layer's result kept and
    the weighted sum over all results, then the next norm; every option off and on."""
    from chibillm_b200.kernels.ops import PendingSum
    g = torch.Generator().manual_seed(T + n + splits)
    x, parts = torch.randn(T, n, generator=g), torch.randn(splits, T, n, generator=g)
    vec, bias = torch.rand(n, generator=g) + 0.2, torch.randn(n, generator=g)
    w = (0.5 + torch.rand(n, generator=g)).to(DTYPES[dtype])
    held = torch.randn(4, T, n, generator=g)
    coeff = torch.randn(4, generator=g)
    for eps, b, depth, norm in ((1e-5, bias, 3, True), (None, None, None, False), (1e-3, None, 4, True), (1e-5, bias, 1, False),
                                (None, bias, 2, True), (1e-5, None, None, True)):
        y = parts.double().sum(0) + (0 if b is None else b.double())
        new = x.double() + vec.double() * (y if eps is None else plain.rms_unit(y, eps))
        outputs, res = held.clone().to(DEV), x.clone().to(DEV)
        out = torch.full((T, n), float("nan"), dtype=DTYPES[dtype], device=DEV)
        arg = None
        total = new
        if depth is not None:
            weights = torch.randn(depth + 1, generator=g)
            arg = (outputs, depth, weights.to(DEV))
            total = plain.depth_average([held[j].double() for j in range(depth)] + [new], weights.double())
        delta = parts[0].to(DEV) if splits == 1 else PendingSum(kernels, parts.to(DEV), splits, T, n)
        kernels.sublayer_end(res, delta, vec.to(DEV), eps, None if b is None else b.to(DEV), arg,
                             norm=(w.to(DEV), 1e-5, 0.0, out) if norm else None)
        what = f"sublayer's end {T} {n} {splits} {dtype} {eps} {depth}"
        close(res, total, 3e-6, what)
        if norm:
            close(out, plain.rms_norm(total, w.double(), 1e-5), KTOL[dtype], what + " norm")
        if depth is not None:
            for j in range(4):
                close(outputs[j], new if j == depth else held[j].double(), 3e-6, what + f" kept {j}")


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("n,top", [(8, 2), (5, 5), (33, 1), (130, 8), (1, 1)])
def test_sigmoid_router(kernels, n, top):
    g = torch.Generator().manual_seed(n * top)
    T = 257
    logits = torch.randn(T, n + 1, generator=g) * 1.5               # one more column, which is not the router's
    w = {"r.router": torch.eye(n, dtype=torch.float64)}
    margins = torch.full((T,), float("inf"), dtype=torch.float64)
    ref_chosen, ref_weight = plain.route(logits[:, :n].double(), top, w, "r.", margins)
    chosen = torch.empty(T, top, dtype=torch.int32, device=DEV)
    share = torch.empty(T, top, dtype=torch.float32, device=DEV)
    kernels.router_choose(logits.to(DEV)[:, :n], None, chosen, share, 1, 1, 1.0, sigmoid=True)
    clear = margins > 1e-6
    assert int(clear.sum()) > T * 0.9
    order = torch.sort(chosen.cpu().long(), 1)
    want = torch.sort(ref_chosen, 1)
    assert torch.equal(order.values[clear], want.values[clear])
    close(share.cpu().gather(1, order.indices)[clear], ref_weight.gather(1, want.indices)[clear], 1e-6, "router weights")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,D,F,E,top", [(1, 64, 24, 6, 2), (9, 48, 16, 4, 1), (300, 96, 40, 5, 4), (700, 128, 64, 7, 2),
                                         (64, 256, 128, 8, 3), (5, 352, 160, 12, 1), (1500, 256, 64, 3, 2), (40, 72, 24, 5, 3)])
def test_experts_with_weighted_inputs_beside_a_gated_one(kernels, dtype, T, D, F, E, top):
    """sum over a token's choices of expert(weight * x), + sigmoid(gate) * base (one array or partial sums), written
    over the accumulator or added to it; plain, mma.sync and tcgen05 kernels by size."""
    from chibillm_b200.kernels.ops import PendingSum
    g = torch.Generator().manual_seed(T + D + F)
    dt = DTYPES[dtype]
    x = torch.randn(T, D, generator=g)
    chosen = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    share = torch.rand(T, top, generator=g)
    gate, up = torch.randn(E, F, D, generator=g) * 1.5 / math.sqrt(D), torch.randn(E, F, D, generator=g) / math.sqrt(D)
    down = torch.randn(E, D, F, generator=g) * 2 / math.sqrt(F)
    base, base_gate = torch.randn(3, T, D, generator=g), torch.randn(T, E + 1, generator=g)
    xd = rounded(x, dtype)
    ref = torch.zeros(T, D, dtype=torch.float64)
    w = {}
    for e_ in range(E):
        w.update({f"e{e_}.gate": rounded(gate[e_], dtype), f"e{e_}.up": rounded(up[e_], dtype),
                  f"e{e_}.down": rounded(down[e_], dtype)})
        rows = (chosen == e_).nonzero()
        if rows.numel():
            weight = share[rows[:, 0], rows[:, 1]].double()[:, None]
            ref.index_add_(0, rows[:, 0], plain.expert_ff(weight * xd[rows[:, 0]], w, f"e{e_}."))
    inter = kernels.expert_tensor_cores(dt, D, F)
    stacked = torch.stack([kernels.interleave_expert_gate_up(gate[e_].to(dt), up[e_].to(dt)) if inter
                           else torch.cat([gate[e_], up[e_]]).to(dt) for e_ in range(E)])
    pairs = T * top
    for splits, overwrite in ((1, True), (3, True), (1, False), (0, True), (0, False)):
        acc = torch.full((T, D), 100.0 if overwrite else 1.0, device=DEV)
        want = ref + (0.0 if overwrite else 1.0)
        extra = {}
        gates = base_gate.to(DEV)
        if splits:
            want = want + torch.sigmoid(base_gate[:, E:].double()) * base[:splits].double().sum(0)
            b = base[0].to(DEV) if splits == 1 else PendingSum(kernels, base.to(DEV), 3, T, D)
            extra["base"] = (b, gates[:, E:])
        route = torch.empty(kernels.route_words(pairs, E), dtype=torch.int32, device=DEV)
        act = torch.empty(pairs, F, dtype=dt, device=DEV)
        y = torch.empty(pairs, D, dtype=torch.float32, device=DEV)
        sorted_x = torch.empty(pairs, D, dtype=dt, device=DEV)
        kernels.chosen_experts(x.to(dt).to(DEV), chosen.to(torch.int32).to(DEV), share.to(DEV), stacked.to(DEV),
                               down.to(dt).to(DEV), acc, route, act, y, "silu", sorted_x, gated=True, interleaved=inter,
                               weight_on_input=True, overwrite=overwrite, **extra)
        kernels.check_error_word()
        close(acc, want, KTOL[dtype] * 2, f"experts {T} {D} {F} {E} {top} {dtype} {splits} {overwrite}")


# ------------------------------------------------------------------ whole models
SEED = 21
CASES = {"P1": (4, [1, 40, 100], [20, 70, 9, 130, 33, 2, 64]),
         "P2": (16, [2, 64, 90], [20, 70, 9, 100, 33, 2]),
         "P3": (16, [3, 70, 150], [150, 64, 9, 200, 33, 2, 100]),
         "P4": (8, [5, 33, 120], [20, 70, 9, 130, 33, 2, 64])}
TOL = {"float32": helpers.TOL["float32"], "bfloat16": 1e-2}


def weights_for(config, dtype, seed=SEED):
    w = pafivik_models.random_weights(config, seed)
    return pafivik_models.decisive(w) if dtype == "bfloat16" else w


def make_runner(folder, dtype, page_size, pool_tokens, max_requests=4):
    from chibillm_b200.engine.runner import ModelRunner
    runner = ModelRunner.from_folder(folder, dtype=dtype, device=DEV, page_size=page_size,
                                     pool_tokens=pool_tokens, max_requests=max_requests)
    runner.storage.poison()
    return runner


def compare(got, ref, margins, dtype, what):
    a, b = pafivik_models.cut_to_safe(got, ref, margins, dtype, most_lost=0.7 if dtype == "float32" else 0.1)
    helpers.assert_logits_close(pafivik_models.without_common_part(a), pafivik_models.without_common_part(b), TOL[dtype],
                                what)


ALONE = {
    "delta rule": pafivik_models.channel_delta(4, 2, 32, 48, conv=3, ranks=(8, 16)),
    "delta rule, values smaller than keys": pafivik_models.channel_delta(3, 1, 20, 12, conv=4, ranks=(3, 9)),
    "linear attention": pafivik_models.lightning(4, 32, 32, decay=[0.5, 0.9, 0.99, 1.0]),
    "linear attention, other value size": pafivik_models.lightning(3, 20, 36),
    "attention": pafivik_models.attention(4, 2, 32, 32, rot=16, base=1000.0),
    "attention, other value size": pafivik_models.attention(6, 2, 16, 24, rot=16),
    "dense": pafivik_models.attention(1, 1, 16, mlp=pafivik_models.dense(72)),
    "experts": pafivik_models.attention(1, 1, 16, mlp=pafivik_models.moe(64, 6, 2, shared=32)),
    "experts, none shared": pafivik_models.attention(1, 1, 16, mlp=pafivik_models.moe(24, 4, 3)),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(ALONE))
def test_one_layer_alone(tmp_path, kind, dtype):
    cfg = {"architecture": "Pafivik", "vocab": 101, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 2.0,
           "layers": [ALONE[kind]]}
    w = weights_for(cfg, dtype, 7)
    folder = pafivik_models.write_model(cfg, str(tmp_path / "one"), seed=7, weights=w)
    reqs = helpers.random_requests(cfg["vocab"], [1, 30, 130], seed=3)
    margins = {}
    ref = pafivik_models.plain_logits(cfg, 7, reqs, weights=w, margins=margins)
    runner = make_runner(folder, dtype, 16, 192)
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (helpers.trace_last_decoded(reqs, 40), "decoded"),
                        (helpers.trace_portions(reqs, seed=5), "portions")):
        compare(helpers.run_trace(runner, trace), ref, margins, dtype, f"pafivik one layer ({kind}) {dtype} {what}")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("pafivik")
    return {(name, dtype): pafivik_models.write_model(pafivik_models.get(name), str(root / f"{name}_{dtype}"), seed=SEED,
                                                      weights=weights_for(pafivik_models.get(name), dtype))
            for name in CASES for dtype in DTYPES}


@pytest.fixture(scope="module")
def expected():
    out = {}
    for name, (_, lengths, mixed_lengths) in CASES.items():
        for dtype in DTYPES:
            cfg = pafivik_models.get(name)
            w = weights_for(cfg, dtype)
            reqs = helpers.random_requests(cfg["vocab"], lengths, seed=100)
            mixed = helpers.random_requests(cfg["vocab"], mixed_lengths, seed=200)
            m1, m2 = {}, {}
            out[name, dtype] = (reqs, pafivik_models.plain_logits(cfg, SEED, reqs, weights=w, margins=m1), m1,
                                mixed, pafivik_models.plain_logits(cfg, SEED, mixed, weights=w, margins=m2), m2)
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(CASES))
def test_cutting_and_batching(folders, expected, case, dtype):
    page_size, lengths, _ = CASES[case]
    reqs, ref, margins, mixed_reqs, mixed_ref, mixed_margins = expected[case, dtype]
    runner = make_runner(folders[case, dtype], dtype, page_size, pool_tokens=helpers.round64(max(lengths)))
    for trace, what in ((helpers.trace_whole(reqs), "whole"),
                        (helpers.trace_last_decoded(reqs, 32), "last 32 decoded"),
                        (helpers.trace_portions(reqs, seed=2), "portions")):
        got = helpers.run_trace(runner, trace)
        compare(got, ref, margins, dtype, f"pafivik {case} {dtype} {what}")
        runner.cache.check_invariants()
        assert not runner.cache.requests
    runner.runtime.kernels.check_error_word()
    pool = 384
    trace = helpers.trace_mixed(mixed_reqs, pool, seed=6)
    assert sum(helpers.round64(len(v)) for v in mixed_reqs.values()) > pool       # pages and slots are used again
    runner2 = make_runner(folders[case, dtype], dtype, page_size, pool)
    got = helpers.run_trace(runner2, trace)
    compare(got, mixed_ref, mixed_margins, dtype, f"pafivik {case} {dtype} mixed")
    runner2.cache.check_invariants()
    assert not runner2.cache.requests


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sublayers_that_add_into_a_zeroed_array(folders, expected, dtype, monkeypatch):
    """The same model with every part adding its result instead of writing it."""
    from chibillm_b200.parts import attention, channel_delta, linear_attention, mlp
    reqs, ref, margins = expected["P3", dtype][:3]
    for part in (attention.PagedAttention, channel_delta.ChannelDelta, linear_attention.LinearAttention, mlp.DenseMLP,
                 mlp.RoutedExperts):
        monkeypatch.setattr(part, "can_overwrite", False)
    runner = make_runner(folders["P3", dtype], dtype, 16, 192)
    compare(helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 20)), ref, margins, dtype,
            f"pafivik P3 {dtype}, sublayers added")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_against_each_request_alone(folders, dtype):
    """Four unequal requests in the same steps against each in steps of its own, both against the plain
    implementation."""
    cfg = pafivik_models.get("P3")
    w = weights_for(cfg, dtype)
    reqs = helpers.random_requests(cfg["vocab"], [90, 7, 140, 33], seed=17)
    margins = {}
    ref = pafivik_models.plain_logits(cfg, SEED, reqs, weights=w, margins=margins)
    runner = make_runner(folders["P3", dtype], dtype, 16, 512)
    alone = helpers.run_trace(runner, helpers.trace_portions(reqs, seed=3))
    compare(alone, ref, margins, dtype, f"pafivik P3 {dtype} each alone")
    steps, pos = [], {r: 0 for r in reqs}
    sizes = {"r0": 13, "r1": 1, "r2": 40, "r3": 2}
    while any(pos[r] < len(ids) for r, ids in reqs.items()):
        entries, end = [], []
        for r, ids in reqs.items():
            if pos[r] < len(ids):
                n = min(sizes[r], len(ids) - pos[r])
                entries.append({"id": r, "tokens": ids[pos[r]:pos[r] + n], "want": list(range(n))})
                pos[r] += n
                if pos[r] == len(ids):
                    end.append(r)
        steps.append({"step": len(steps), "entries": entries, "end": end})
    together = helpers.run_trace(runner, steps)
    compare(together, ref, margins, dtype, f"pafivik P3 {dtype} together")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_whole_and_in_portions(folders, dtype):
    """1,100 tokens through the model of tensor-core sizes: whole, in portions of about 100 tokens and with its
    last 40 tokens decoded."""
    cfg = pafivik_models.get("P3")
    w = weights_for(cfg, "bfloat16")
    reqs = helpers.random_requests(cfg["vocab"], [1100], seed=31)
    margins = {}
    ref = pafivik_models.plain_logits(cfg, SEED, reqs, weights=w, margins=margins)
    runner = make_runner(folders["P3", "bfloat16"], dtype, 16, 1152)
    ids = reqs["r0"]
    steps, pos, sizes, k = [], 0, [100, 130, 128, 3, 117], 0
    while pos < len(ids):
        n = min(sizes[k % len(sizes)], len(ids) - pos)
        k += 1
        steps.append({"step": len(steps), "entries": [{"id": "r0", "tokens": ids[pos:pos + n], "want": list(range(n))}],
                      "end": ["r0"] if pos + n == len(ids) else []})
        pos += n
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (steps, "portions of about 100"),
                        (helpers.trace_last_decoded(reqs, 40), "last 40 decoded")):
        compare(helpers.run_trace(runner, trace), ref, margins, dtype, f"pafivik P3 {dtype} long prompt {what}")
    runner.runtime.kernels.check_error_word()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    """Three tokens of prompt, then 300 tokens one by one (captured steps replayed): the states and the
    convolution's history are carried 300 times."""
    cfg = pafivik_models.get("P1")
    w = weights_for(cfg, "bfloat16")
    reqs = helpers.random_requests(cfg["vocab"], [303], seed=9)
    margins = {}
    ref = pafivik_models.plain_logits(cfg, SEED, reqs, weights=w, margins=margins)
    runner = make_runner(folders["P1", "bfloat16"], dtype, 4, 320)
    got = helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 300))
    compare(got, ref, margins, dtype, f"pafivik P1 {dtype} long decoding")
    assert runner.graph_replays > 200


def test_greedy_generation_through_the_entry_point(folders):
    """``LLM.generate`` (scheduler, sampler, portions of 16 tokens, three requests at a time): every generated
    token is the plain implementation's best one, wherever that leads by more than the rounding of a 32-bit
    run and no router's choice was a close call."""
    from chibillm_b200 import LLM
    cfg = pafivik_models.get("P3")
    w = pafivik_models.decisive(pafivik_models.random_weights(cfg, SEED))
    prompts = list(helpers.random_requests(cfg["vocab"], [5, 40, 23, 61], seed=12).values())
    llm = LLM(folders["P3", "bfloat16"], dtype="float32", context_length=128, max_sequences=3, max_batch_tokens=48,
              prefill_chunk_tokens=16, page_size=16)
    outs = llm.generate(prompts, max_tokens=12, ignore_eos=True)
    for prompt, new in zip(prompts, outs):
        assert len(new) == 12
        ref = pafivik_models.plain_logits(cfg, SEED, {"a": prompt + new}, weights=w)["a"]
        for i, tok in enumerate(new):
            row = ref[len(prompt) + i - 1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(row.abs().max()):
                assert int(torch.argmax(row)) == tok, f"token {i} of a prompt of {len(prompt)}"


def test_trace_program(folders, tmp_path):
    """bin/trace_run on a Pafivik folder: portions, single tokens, two live requests."""
    a_len, b_len = 40, 21
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = pafivik_models.get("P4")
    w = weights_for(cfg, "bfloat16")
    reqs = helpers.random_requests(cfg["vocab"], [a_len, b_len], seed=5)
    ref = pafivik_models.without_common_part(pafivik_models.plain_logits(cfg, SEED, reqs, weights=w))
    a, b = reqs["r0"], reqs["r1"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]},
                                     {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[19:], "want": [0, 1]},
                                     {"id": "a", "tokens": a[31:], "want": [8]}], "end": ["a", "b"]}]
    want = [[("r0", 0), ("r0", 29)], [("r0", 30), ("r1", 18)], [("r1", 19), ("r1", 20), ("r0", 39)]]
    for dtype in ("float32", "bfloat16"):
        out_dir = str(tmp_path / dtype)
        proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model",
                               folders["P4", "bfloat16"], "--dtype", dtype, "--out", out_dir, "--max-tokens", "128"],
                              input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                              timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        for i, rows in enumerate(want):
            got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(len(rows), -1))
            for j, (r, pos) in enumerate(rows):
                scale = float(ref[r].abs().max())
                diff = (got[j] - got[j].mean()) - ref[r][pos]
                assert float(diff.abs().max()) <= TOL[dtype] * scale, (dtype, i, r, pos)


def test_random_weights_made_on_the_device(tmp_path):
    """``ModelRunner.from_random`` makes on the device the values that ``write_random_model`` stores: both
    give the same logits."""
    from chibillm_b200.engine.batch import StepEntry
    from chibillm_b200.engine.runner import ModelRunner
    from chibillm_b200.weights import write_random_model
    cfg = pafivik_models.with_rank_keys(pafivik_models.get("P4"))
    folder = write_random_model(cfg, str(tmp_path / "random"), seed=6)
    ids = helpers.random_requests(cfg["vocab"], [50], seed=2)["r0"]
    a = ModelRunner.from_folder(folder, dtype="float32", device=DEV, page_size=8, pool_tokens=64)
    b = ModelRunner.from_random(cfg, seed=6, dtype="float32", device=DEV, page_size=8, pool_tokens=64)
    la = a.step([StepEntry("x", ids, list(range(50)))]).clone()
    lb = b.step([StepEntry("x", ids, list(range(50)))]).clone()
    assert torch.equal(la, lb)
