"""Lefavik on the GPU against the plain implementation of the design (tests/plain_lefavik.py): each mechanism's
kernels alone -- learned positions with the norm behind them; heads with a unit norm and a temperature, from an
array and from a product's partial sums; attention with a distance bias, a window and one added to the
denominator, keys made to stand out just inside and just outside the window, at page borders, in prompts and for
tokens decoded alone; the queries, cache rows and gates of latent attention, one far key among hundreds and a sink
as heavy as it; gated products with the tanh form of gelu; two last products side by side -- then one layer of each
kind alone and whole models through the step function: whole prompts, the last tokens one by one, portions down to
two tokens, mixed batches with reused pages, long prompts and long decoding; then greedy generation through the
package's entry point and the trace program."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import helpers
import lefavik_models
import plain_lefavik as plain

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


def as_product(kernels, x, splits, dtype):
    """Rows [T, n] as the kernel after a product gets them: an array of the activations' type, or partial sums.
    Returns that and the rows' values in 64-bit."""
    from chibillm_b200.kernels.ops import PendingSum
    if splits == 1:
        return x.to(DTYPES[dtype]).to(DEV), rounded(x, dtype)
    parts = torch.randn(splits, *x.shape, generator=torch.Generator().manual_seed(splits)) * 0.3
    parts[-1] += x
    return PendingSum(kernels, parts.to(DEV), splits, *x.shape), parts.double().sum(0)


def scrambled_table(tokens, page_size, seed=0):
    """(block table on the device whose row 1 is a sequence's, its pages in order, number of pages)."""
    pages = (tokens + page_size - 1) // page_size + 3
    given = torch.randperm(pages, generator=torch.Generator().manual_seed(seed + tokens))[:pages - 3]
    table = torch.full((2, pages), -1, dtype=torch.int32)
    table[1, :given.numel()] = given.to(torch.int32)
    return table.to(DEV), given, pages


# ------------------------------------------------------------------ the start and the ends of a layer
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,n", [(1, 48), (37, 70), (300, 256), (5, 1001), (3, 5000), (65, 4096)])
def test_position_rows(kernels, dtype, T, n):
    g = torch.Generator().manual_seed(T + n)
    x, table = torch.randn(T, n, generator=g), torch.randn(50, n, generator=g)
    w = 0.5 + torch.rand(n, generator=g)
    pos = torch.randint(0, 50, (T,), generator=g)
    pos[0], pos[-1] = 49, 0
    for factor, weight, eps in ((2.5, w, 1e-5), (-0.3, None, 0.0), (1.0, w, 0.7)):
        ref = factor * x.double() + rounded(table, dtype)[pos]
        if weight is not None:
            ref = plain.unit_rms(ref, eps) * weight.double()
        got = x.clone().to(DEV)
        kernels.position_rows(got, factor, table.to(DTYPES[dtype]).to(DEV), pos.to(torch.int32).to(DEV),
                              None if weight is None else weight.to(DEV), eps)
        close(got, ref, 2e-6, f"position rows {T} {n} {dtype} {factor}")
    kernels.check_error_word()


def test_a_position_outside_the_table_is_reported(kernels):
    from chibillm_b200.kernels.ops import KernelError
    x = torch.ones(3, 16, device=DEV)
    for bad in (5, -1):
        kernels.position_rows(x, 1.0, torch.ones(5, 16, device=DEV), i32([0, bad, 4]), None, 0.0)
        with pytest.raises(KernelError, match="position"):
            kernels.check_error_word()
    kernels.check_error_word()


@pytest.mark.parametrize("T", [1, 8, 17, 64, 65, 200, 700, 2048])
@pytest.mark.parametrize("D,F", [(64, 64), (256, 320), (512, 1024), (1024, 3072)])
def test_gated_products_with_gelu(kernels, T, D, F):
    """gelu_tanh(x gate^T) * (x up^T) in one product for few and many rows, arguments from tiny to far out on both
    sides; silu by the same kernels beside it."""
    g = torch.Generator().manual_seed(T + D)
    x = torch.randn(T, D, generator=g).to(torch.bfloat16)
    gate = (torch.randn(F, D, generator=g) * torch.logspace(-1, 1, F)[:, None] / math.sqrt(D)).to(torch.bfloat16)
    up = (torch.randn(F, D, generator=g) / math.sqrt(D)).to(torch.bfloat16)
    z, u = x.double() @ gate.double().T, x.double() @ up.double().T
    w = kernels.interleave_gate_up(gate.to(DEV), up.to(DEV))
    assert w is not None
    for kind, ref in (("gelu_tanh", plain.gelu_tanh(z) * u), ("silu", z * torch.sigmoid(z) * u)):
        out = torch.full((T, F), float("nan"), dtype=torch.bfloat16, device=DEV)
        assert kernels.linear_swiglu(x.to(DEV), w, out, **({} if kind == "silu" else {"kind": kind}))
        err = (out.double().cpu() - ref).abs()
        bound = 6e-3 * ref.abs() + 2e-5 * (1 + z.abs()) * (1 + u.abs())       # of every value by itself
        assert bool((err <= bound).all()), (kind, T, D, F, float((err / bound).max()))
    kernels.check_error_word()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,N,K1,K2", [(1, 1024, 1024, 3072), (8, 64, 72, 40), (8, 2048, 4096, 6144), (17, 72, 200, 320),
                                       (33, 131, 64, 512), (64, 512, 2048, 256), (65, 256, 128, 512), (300, 1024, 512, 2048)])
def test_two_products_side_by_side(kernels, dtype, T, N, K1, K2):
    g = torch.Generator().manual_seed(T + N)
    dt = DTYPES[dtype]
    x1, x2 = torch.randn(T, K1, generator=g).to(dt), torch.randn(T, K2, generator=g).to(dt)
    w1 = (torch.randn(N, K1, generator=g) / math.sqrt(K1)).to(dt)
    w2 = (torch.randn(N, K2, generator=g) / math.sqrt(K2)).to(dt)
    res = torch.randn(T, N, generator=g)
    ref = res.double() + x1.double() @ w1.double().T + x2.double() @ w2.double().T
    got = res.clone().to(DEV)
    left = kernels.linear_pair(x1.to(DEV), w1.to(DEV), x2.to(DEV), w2.to(DEV), got)
    if left is not None:
        left.add_into(got)
    close(got, ref, 1e-5, f"two products {T} {N} {K1} {K2} {dtype}")
    kernels.check_error_word()


def test_a_factor_per_row_is_applied_once_for_two_readers(kernels):
    """A norm's output whose factor per row is still to be applied, read by two products of which the first (or
    the second) cannot apply it itself: the array gets the factor once."""
    g = torch.Generator().manual_seed(1)
    T, D = 300, 256
    x, res = torch.randn(T, 512, generator=g).to(torch.bfloat16), torch.randn(T, D, generator=g)
    w0 = (torch.randn(D, 512, generator=g) / 22).to(torch.bfloat16)
    nw = (0.5 + torch.rand(D, generator=g)).to(torch.bfloat16)
    odd, even = ((torch.randn(n, D, generator=g) / 16).to(torch.bfloat16) for n in (72, 256))
    h = res.double() + x.double() @ w0.double().T
    normed = plain.unit_rms(h, 1e-5) * nw.double()
    for order in ((odd, even), (even, odd), (odd, odd), (even, even)):
        r = res.clone().to(DEV)
        out = torch.empty(T, D, dtype=torch.bfloat16, device=DEV)
        rows = kernels.linear_residual_norm(x.to(DEV), w0.to(DEV), r, nw.to(DEV), 1e-5, 0.0, out)
        assert rows is not None
        for w in order:
            y = torch.empty(T, w.shape[0], dtype=torch.bfloat16, device=DEV)
            kernels.linear(rows, w.to(DEV), y)
            close(y, normed @ w.double().T, 2e-2, f"reader of {w.shape[0]} columns")


# ------------------------------------------------------------------ attention in a window
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,e", [(6, 3, 16, 16), (4, 1, 20, 33), (5, 5, 48, 16), (6, 2, 10, 7), (8, 2, 128, 128), (3, 3, 200, 64)])
def test_heads_with_a_unit_norm_and_a_temperature(kernels, dtype, H, G, d, e):
    """q, k and v of single tokens at chosen positions (steps of the temperature, both sides), from an array and
    from partial sums; what no option asks for stays as it was."""
    g = torch.Generator().manual_seed(d + e)
    dt = DTYPES[dtype]
    page, T = 8, 70
    table, given, pages = scrambled_table(T, page)
    x = torch.randn(T, H * d + G * d + G * e, generator=g) * torch.logspace(-2, 1, T)[:, None]
    for splits in ((1,) if dtype == "float32" else (1, 2, 5, 9)):
        for eps, temp in ((1e-5, (0.4, 7)), (1e-3, (-0.2, 1)), (0.5, None), (None, (1.5, 64)), (None, None)):
            rows, values = as_product(kernels, x, splits, dtype)
            kc = torch.full((pages, G, page, d), 9.0, dtype=dt, device=DEV)
            vc = torch.full((pages, G, page, e), 9.0, dtype=dt, device=DEV)
            q_out = torch.empty(T, H * d, dtype=dt, device=DEV)
            kernels.heads_prepare_append(rows, q_out, kc, vc, None, None, None, 0.0, None, 0, i32(list(range(T))),
                                         i32([0] * T), table, H, G, G, d, e, page, i32([1]), unit_norm_eps=eps,
                                         temperature=temp)
            q, k, v = values[:, :H * d].view(T, H, d), values[:, H * d:(H + G) * d].view(T, G, d), values[:, (H + G) * d:]
            if eps is not None:
                q, k = plain.unit_rms(q, eps), plain.unit_rms(k, eps)
            if temp is not None:
                q = q * plain.temperature(T, *temp)[:, None, None]
            tol = 2e-6 if dtype == "float32" else 4e-3
            for t in (0, 1, 5, 6, 7, 13, 62, 63, 64, T - 1):           # (each row by its own size)
                where = (given[t // page].item(), slice(None), t % page)
                close(q_out[t].view(H, d), q[t], tol, f"q of {t}, {splits} {eps} {temp}")
                close(kc[where], k[t], tol, f"k of {t}, {splits} {eps} {temp}")
                close(vc[where], v[t].view(G, e), tol, f"v of {t}, {splits} {eps} {temp}")
            unused = [p for p in range(pages) if p not in given.tolist()]
            assert float((kc[unused].float() - 9.0).abs().max()) == 0.0 == float((vc[unused].float() - 9.0).abs().max())
    kernels.check_error_word()


def run_window_attention(kernels, q, k, v, m, eps, dtype, page_size, portions):
    """q [T, H, d], k [T, G, d], v [T, G, e] of one sequence through the two kernels of the mixer."""
    dt = DTYPES[dtype]
    T, H, d = q.shape
    G, e = k.shape[1], v.shape[2]
    table, _, pages = scrambled_table(T, page_size)
    kc = torch.full((pages, G, page_size, d), float("nan"), dtype=dt, device=DEV)
    vc = torch.full((pages, G, page_size, e), float("nan"), dtype=dt, device=DEV)
    row = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1)], 1).to(dt).to(DEV)
    temp = (m["q_temp"]["coef"], m["q_temp"]["every"]) if m.get("q_temp") else None
    size = (m.get("mask") or {}).get("size")
    slopes = plain.slopes(H).float().to(DEV)
    outs, pos = [], 0
    for n in portions:
        n = min(n, T - pos)
        if n <= 0:
            break
        positions, seq_of, rows = i32(list(range(pos, pos + n))), i32([0] * n), i32([1])
        q_out = torch.empty(n, H * d, dtype=dt, device=DEV)
        kernels.heads_prepare_append(row[pos:pos + n], q_out, kc, vc, None, None, None, 0.0, None, 0, positions, seq_of,
                                     table, H, G, G, d, e, page_size, rows, unit_norm_eps=eps, temperature=temp)
        out = torch.empty(n, H * e, dtype=dt, device=DEV)
        kernels.attention(q_out, kc, vc, out, table, i32([0, n]), i32([pos + n]), seq_of, positions, H, G, d, page_size,
                          m["scale"], size, n, pos + n, n, rows, value_dim=e, sink=torch.zeros(H, device=DEV),
                          distance_bias=(slopes, None))
        outs.append(out.float().cpu().view(n, H, e))
        pos += n
    kernels.check_error_word()
    return torch.cat(outs)


def plain_window_attention(q, k, v, m, eps, dtype):
    """The mixer without its projections, on inputs rounded as the kernels' are."""
    T, H, d = q.shape
    G, e = k.shape[1], v.shape[2]
    x = torch.cat([rounded(t, dtype).reshape(T, -1) for t in (q, k, v)], 1)
    w = {"q": torch.eye(x.shape[1], dtype=torch.float64)[:H * d],
         "k": torch.eye(x.shape[1], dtype=torch.float64)[H * d:(H + G) * d],
         "v": torch.eye(x.shape[1], dtype=torch.float64)[(H + G) * d:],
         "o": torch.eye(H * e, dtype=torch.float64)}
    return plain.window_attention(x, dict(m, heads=H, kv_heads=G, dim=d, vdim=e), w, "", eps).view(T, H, e)


WINDOW_CUTS = ([10000], [40, 2, 1, 1, 70, 3, 33, 2, 150], [100] + [1] * 400)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,e,size,temp", [
    (6, 3, 16, 16, 5, (0.4, 7)), (4, 1, 20, 33, 16, None), (6, 2, 10, 7, 1, (1.3, 3)), (8, 2, 64, 64, 100, (0.05, 1)),
    (4, 4, 128, 128, 64, None), (5, 5, 48, 16, 17, (0.3, 16)), (3, 1, 48, 48, 129, (0.2, 128)), (12, 2, 80, 80, None, (0.1, 30)),
    (2, 2, 128, 128, None, None), (4, 2, 32, 64, 33, None)])
def test_attention_with_distance_window_and_one_added(kernels, dtype, H, G, d, e, size, temp):
    g = torch.Generator().manual_seed(d * 7 + e)
    T = 260
    q, k, v = torch.randn(T, H, d, generator=g), torch.randn(T, G, d, generator=g), torch.randn(T, G, e, generator=g)
    m = {"scale": 3.0 / math.sqrt(d)}
    if size is not None:
        m["mask"] = {"size": size}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    ref = plain_window_attention(q, k, v, m, 1e-5, dtype)
    for portions in WINDOW_CUTS:
        got = run_window_attention(kernels, q, k, v, m, 1e-5, dtype, 16, portions)
        close(got, ref, KTOL[dtype], f"window attention {H} {G} {d} {e} {size} {temp} {dtype} {portions[:2]}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("d,e,size", [(16, 16, 33), (64, 64, 100), (128, 128, 64), (24, 10, 40), (48, 16, 17)])
def test_the_windows_edge_and_the_added_one(kernels, dtype, d, e, size):
    """One key stands out (its score beats the others' by far, its value is known).  The last query that is to see
    it returns its value times score / (1 + score), as exp(score) against the added one demands; the next
    query returns next to nothing of it.  The key sits at the start, at page borders and far from them."""
    H, G, T, page = 2, 1, 420, 16
    m = {"scale": 1.0 / d, "mask": {"size": size}}
    for key_pos in (0, 15, 16, 207, 240):
        g = torch.Generator().manual_seed(key_pos)
        base = torch.randint(0, 2, (d,), generator=g).double() * 2 - 1
        other = base.clone()
        other[::2] *= -1                                            # orthogonal to it (d even)
        q = (6.0 * base).float().expand(T, H, d).contiguous()
        k = other.float().expand(T, G, d).contiguous().clone()
        k[key_pos] = base.float()
        v = torch.zeros(T, G, e)
        v[key_pos] = 7.0
        # unit norms: q . k = d for the marked key, 0 for others: scores scale * d = 1 less the distance; scaled up
        m["scale"] = 12.0 / d
        ref = plain_window_attention(q, k, v, m, 1e-6, dtype)
        last = key_pos + size - 1
        assert float(ref[last, 1].min()) > 0.5 and float(ref[last + 1].abs().max()) == 0.0
        for portions in ([T], [key_pos + size - 2 if key_pos + size > 2 else 1] + [1] * 6 + [T], [last + 1, 2, T], [3, 2, 290, 2, 1, 1, 1, 2, 200]):
            got = run_window_attention(kernels, q, k, v, m, 1e-6, dtype, page, portions)
            close(got[last], ref[last], KTOL[dtype], f"just inside, {d} {size} key {key_pos}")
            assert float(got[last + 1].abs().max()) < 1e-4, (d, size, key_pos)
            close(got, ref, KTOL[dtype], f"all rows, {d} {size} key {key_pos}")
    # without scores at all: a first token keeps half its value (exp(0) against the added one)
    z = torch.zeros(3, H, d)
    got = run_window_attention(kernels, z, torch.zeros(3, G, d), torch.ones(3, G, e), {"scale": 1.0}, 1e-5, dtype, page, [3])
    assert float((got[0] - 0.5).abs().max()) < 1e-3


# ------------------------------------------------------------------ latent attention
LATENT_SHAPES = [(4, 40, 8), (5, 27, 6), (2, 20, 4), (8, 96, 32), (6, 128, 64), (3, 256, 64), (32, 192, 64), (1, 700, 66)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,c,r", LATENT_SHAPES)
def test_queries_cache_rows_and_gates(kernels, dtype, H, c, r):
    """From an array (wider than what is read) and from partial sums; with and without a cache and gates; positions
    that start inside a page."""
    g = torch.Generator().manual_seed(H + c + r)
    dt = DTYPES[dtype]
    T, first, page, eps, base = 21, 13, 8, 1e-4, 300.0
    kd = c + r
    table, given, pages = scrambled_table(first + T, page)
    norm = 0.5 + torch.rand(c, generator=g)
    freq = torch.tensor([base ** (-2.0 * i / r) for i in range(r // 2)], dtype=torch.float64)
    order = list(range(0, r, 2)) + list(range(1, r, 2))              # the kernels' order of neighbouring pairs
    positions = torch.arange(first, first + T)

    def turn(x):                                                     # [T, heads, r], features in the stored order
        pad = torch.zeros(first, *x.shape[1:], dtype=torch.float64)
        return plain.rotate_neighbours(torch.cat([pad, x]), base, r)[first:]

    x = torch.randn(T, H * kd + kd + H + 5, generator=g)
    for splits in ((1,) if dtype == "float32" else (1, 3, 6)):
        for append, gated in ((True, True), (False, True), (True, False), (False, False)):
            rows, v = as_product(kernels, x, splits, dtype)
            q_out = torch.empty(T, H * kd, dtype=dt, device=DEV)
            cache = torch.full((pages, 1, page, kd), 9.0, dtype=dt, device=DEV)
            gates = torch.full((T, H), float("nan"), device=DEV) if gated else None
            kernels.latent_heads_append(rows, q_out, cache if append else None, norm.to(DEV) if append else None, eps,
                                        freq.float().to(DEV), H, c, r, gates, positions.to(torch.int32).to(DEV), i32([0] * T),
                                        table if append else None, page, i32([1]))
            tol = 2e-5 if dtype == "float32" else 1e-2
            what = f"latent rows {H} {c} {r} {dtype} {splits} {append} {gated}"
            q = v[:, :H * kd].view(T, H, kd)
            back = torch.empty(T, H, r, dtype=torch.float64)
            back[..., order] = q[..., :r]                            # (the rows arrive in the kernels' order)
            want = torch.cat([turn(back)[..., order], q[..., r:]], -1)
            close(q_out.view(T, H, kd), want, tol, what + " q")
            at = H * kd
            if append:
                back = torch.empty(T, 1, r, dtype=torch.float64)
                back[:, 0, order] = v[:, at + c:at + kd]
                want = torch.cat([turn(back)[:, 0][:, order], plain.unit_rms(v[:, at:at + c], eps) * norm.double()], -1)
                got = torch.stack([cache[given[p // page].item(), 0, p % page] for p in positions.tolist()])
                close(got, want, tol, what + " cache row")
                touched = torch.zeros(pages, page, dtype=torch.bool)
                touched[given[positions // page], positions % page] = True
                assert float((cache[:, 0].cpu().float()[~touched] - 9.0).abs().max()) == 0.0
                at += kd
            if gated:
                close(gates, torch.sigmoid(v[:, at:at + H]), 2e-6 if splits == 1 else 1e-5, what + " gates")
    kernels.check_error_word()


@pytest.mark.parametrize("d,H,page", [(144, 3, 8), (160, 2, 32), (192, 8, 16), (208, 5, 16), (224, 1, 8), (256, 32, 16), (256, 6, 32),
                                      (192, 12, 64), (256, 3, 128)])
@pytest.mark.parametrize("window", [None, 100, 1])
def test_prompt_attention_over_rows_that_are_keys_and_values(kernels, d, H, page, window):
    """Several sequences in one step -- a whole prompt, a portion after a long context, two tokens, one token, a
    prompt that fills its last page -- with pages of NaN around what was written; on the kernel for wide rows, and
    (switched off) on the one that it stands for.  A short portion alone after a long context
    runs in key ranges."""
    g = torch.Generator().manual_seed(d + H)
    held = [(0, 300), (1000, 40), (37, 2), (500, 1), (0, 192)]
    T = sum(n for _, n in held)
    pages = sum((c + n + page - 1) // page for c, n in held) + 4
    order = torch.randperm(pages, generator=g).tolist()
    cache = torch.full((pages, 1, page, d), float("nan"), dtype=torch.bfloat16)
    table = torch.full((len(held) + 1, 1200 // page + 2), -1, dtype=torch.int32)
    q = torch.randn(T, H, d, generator=g).to(torch.bfloat16)
    sink, scale = torch.randn(H, generator=g), 3.0 / math.sqrt(d)
    ref, at, starts, seq_of, positions = [], 0, [0], [], []
    for i, (c, n) in enumerate(held):
        rows = torch.randn(c + n, d, generator=g).to(torch.bfloat16)
        for b in range((c + n + page - 1) // page):
            pg = order.pop()
            table[i + 1, b] = pg
            part = rows[b * page:(b + 1) * page]
            cache[pg, 0, :part.shape[0]] = part
        seen = plain.visible(c + n, window)[c:]
        scores = torch.einsum("ihd,jd->hij", q[at:at + n].double(), rows.double()) * scale
        ref.append(torch.stack([plain.weights_with_sink(scores[h], seen, sink[h].double()) @ rows.double() for h in range(H)], 1))
        at += n
        starts.append(at)
        seq_of += [i] * n
        positions += list(range(c, c + n))
    ref = torch.cat(ref).reshape(T, H * d)
    cache, table, qd = cache.to(DEV), table.to(DEV), q.reshape(T, H * d).to(DEV)
    lens = [c + n for c, n in held]

    def run(which, **how):
        lo, hi = starts[which[0]], starts[which[-1] + 1]
        out = torch.full((hi - lo, H * d), float("nan"), dtype=torch.bfloat16, device=DEV)
        ns = [held[i][1] for i in which]
        kernels.attention(qd[lo:hi].contiguous(), cache, cache, out, table, i32([starts[i] - lo for i in which] + [hi - lo]),
                          i32([lens[i] for i in which]), i32([seq_of[t] - which[0] for t in range(lo, hi)]), i32(positions[lo:hi]),
                          H, 1, d, page, scale, window, max(ns), max(lens[i] for i in which), min(ns),
                          i32([i + 1 for i in which]), sink=sink.to(DEV), **how)
        kernels.check_error_word()
        return out, ref[lo:hi]

    for which in ([0, 1, 2, 3, 4], [1], [2], [4], [0]):
        got, want = run(which)
        close(got, want, 2e-2, f"rows of {d}, {H} heads, window {window}, sequences {which}")
    kernels.use_tcgen05_attention = False
    try:
        got, want = run([0, 1, 2, 3, 4])
    finally:
        kernels.use_tcgen05_attention = True
    close(got, want, 2e-2, f"rows of {d} on the other kernel")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,H,n", [(1, 3, 33), (8, 32, 256), (300, 4, 48), (2000, 8, 128), (7, 1, 700)])
def test_head_gate(kernels, dtype, T, H, n):
    g = torch.Generator().manual_seed(T + n)
    x, gates = torch.randn(T, H * n, generator=g), torch.rand(T, H, generator=g)
    got = x.to(DTYPES[dtype]).to(DEV)
    kernels.head_gate(got, gates.to(DEV), H)
    close(got, rounded(x, dtype).view(T, H, n).mul(gates.double()[:, :, None]).reshape(T, -1), 4e-3 if dtype == "bfloat16" else 1e-6,
          "head gate")


# ------------------------------------------------------------------ whole models
SEED = 21
CASES = {"L1": (4, [1, 40, 100], [20, 70, 9, 130, 33, 2, 64]),
         "L2": (16, [2, 64, 90], [20, 70, 9, 100, 33, 2]),
         "L3": (16, [3, 130, 260], [150, 64, 9, 200, 33, 2, 100]),
         "L4": (8, [5, 33, 120], [20, 70, 9, 130, 33, 2, 64])}
TOL = {"float32": helpers.TOL["float32"], "bfloat16": 3e-2}


def make_runner(folder, dtype, page_size, pool_tokens, max_requests=4):
    from chibillm_b200.engine.runner import ModelRunner
    runner = ModelRunner.from_folder(folder, dtype=dtype, device=DEV, page_size=page_size,
                                     pool_tokens=pool_tokens, max_requests=max_requests)
    runner.storage.poison()
    return runner


def model_of(*layers, width=64, positions=1200):
    return {"architecture": "Lefavik", "vocab": 101, "width": width, "max_positions": positions, "norm": {"eps": 1e-5},
            "embedding": {"scale": 3.0}, "logit_scale": 1.5, "layers": list(layers)}


ALONE = {
    "latent": [lefavik_models.latent(4, 24, 8, 20, 40, base=900.0)],
    "latent, cache row of tensor-core size": [lefavik_models.latent(4, 32, 32, 32, 96, base=900.0, ff=64)],
    "latent with a reader": [lefavik_models.latent(4, 16, 16, 24, 48), lefavik_models.latent(6, 8, 16, 12, 48, kv_from=0, ff=40)],
    "window": [lefavik_models.window(6, 2, 32, mask=19, temp=(0.5, 4))],
    "window, values of another size": [lefavik_models.window(4, 2, 16, 48, mask=50, temp=(0.2, 1), ff=72)],
    "no window": [lefavik_models.window(3, 1, 24, 24, ff=128)],
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", list(ALONE))
def test_one_kind_alone(tmp_path, kind, dtype):
    cfg = model_of(*ALONE[kind])
    folder = lefavik_models.write_model(cfg, str(tmp_path / "one"), seed=7)
    reqs = helpers.random_requests(cfg["vocab"], [1, 30, 130], seed=3)
    ref = lefavik_models.plain_logits(cfg, 7, reqs)
    runner = make_runner(folder, dtype, 16, 192)
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (helpers.trace_last_decoded(reqs, 40), "decoded"),
                        (helpers.trace_portions(reqs, seed=5), "portions")):
        helpers.assert_logits_close(helpers.run_trace(runner, trace), ref, TOL[dtype],
                                    f"lefavik one kind ({kind}) {dtype} {what}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [(24, 8, 20, 40), (64, 32, 64, 96), (64, 64, 64, 192)])
def test_a_far_key_and_a_sink_as_heavy(tmp_path, dtype, rows):
    """A latent layer and its reader in which one token of the vocabulary is found by every later query: queries look
    along a direction that only this token's latent has.  It sits far back at page borders; with sinks
    out of reach it takes all weight, with sinks as heavy as its score half of it.  The plain implementation
    with the token replaced shows that the logits depend on it."""
    d, r, e, c = rows
    cfg = model_of(lefavik_models.latent(2, d, r, e, c, scale=1.0), lefavik_models.latent(3, d, r, e, c, scale=1.0, kv_from=0))
    D, T = cfg["width"], 700
    w = {k: v.float() for k, v in lefavik_models.random_weights(cfg, 3).items()}
    w["pos"] *= 0.02
    # feature 0 of the stream: large for token 100 alone; feature 1: the same for all tokens
    w["embed"][:, :2], w["embed"][100, 0], w["embed"][:, 1] = 0.0, 3.0, 1.0
    w["pos"][:, :2] = 0.0
    for i, H in ((0, 2), (1, 3)):
        p = f"l{i}.mix."
        w[p + "q"].zero_()
        w[p + "q"].view(H, d + r, D)[:, 0, 1] = 1.0             # q's first plain feature: feature 1
        w[p + "uk"].zero_()
        w[p + "uk"].view(H, d, c)[:, 0, 0] = 1.0                # k's first plain feature: the latent's first number
        w[p + "o"] *= 3.0
    w["l0.mix.dkv"][0].zero_()
    w["l0.mix.dkv"][0, 0] = 8.0
    ids0 = torch.randint(0, 100, (T,), generator=torch.Generator().manual_seed(2)).tolist()
    stored = lambda ww: {k: v.to(torch.bfloat16) for k, v in ww.items()}

    def score_of(ids, at, ww):
        """The last query's score for the marked key in the first layer."""
        ww = {k: v.double() for k, v in stored(ww).items()}
        h = plain.unit_rms(plain.embed(torch.tensor(ids), cfg, ww), 1e-5) * ww["l0.norm1"]
        latent, _ = plain.latent_rows(h, cfg["layers"][0]["mixer"], ww, "l0.mix.", 1e-5)
        return float((h[-1] @ ww["l0.mix.q"][0]) * (latent[at] @ ww["l0.mix.uk"][0]))

    ids = [100] + ids0[1:]
    gain = 14.0 / score_of(ids, 0, w)                           # exp(14) against hundreds of keys with exp(0)
    for i in (0, 1):
        w[f"l{i}.mix.uk"] *= gain
    for heavy in (False, True):
        for at in (0, 15, 16, 33):
            ids = list(ids0)
            ids[at] = 100
            ww = dict(w)
            for i in (0, 1):
                ww[f"l{i}.mix.sink"] = torch.full_like(w[f"l{i}.mix.sink"], score_of(ids, at, w) if heavy else -30.0)
            ww = stored(ww)
            folder = lefavik_models.write_model(cfg, str(tmp_path / f"{at}_{heavy}"), 3, weights=ww)
            ref = lefavik_models.plain_logits(cfg, 3, {"r0": ids}, weights=ww)
            without = lefavik_models.plain_logits(cfg, 3, {"r0": ids0}, weights=ww)["r0"]
            assert float((ref["r0"][-1] - without[-1]).abs().max()) > 0.1 * float(ref["r0"][-1].abs().max())
            runner = make_runner(folder, dtype, 16, 704, max_requests=1)
            for trace, what in ((helpers.trace_whole({"r0": ids}), "whole"), (helpers.trace_last_decoded({"r0": ids}, 20), "decoded"),
                                (helpers.trace_portions({"r0": ids}, seed=at), "portions")):
                got = helpers.run_trace(runner, trace)
                helpers.assert_logits_close(got, ref, TOL[dtype] * (3 if heavy else 2), f"lefavik far key {rows} heavy {heavy} {dtype} {what}")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("lefavik")
    return {name: lefavik_models.write_model(lefavik_models.get(name), str(root / name), seed=SEED) for name in CASES}


@pytest.fixture(scope="module")
def expected():
    out = {}
    for name, (_, lengths, mixed_lengths) in CASES.items():
        cfg = lefavik_models.get(name)
        reqs = helpers.random_requests(cfg["vocab"], lengths, seed=100)
        mixed = helpers.random_requests(cfg["vocab"], mixed_lengths, seed=200)
        out[name] = (reqs, lefavik_models.plain_logits(cfg, SEED, reqs), mixed, lefavik_models.plain_logits(cfg, SEED, mixed))
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(CASES))
def test_cutting_and_batching(folders, expected, case, dtype):
    page_size, lengths, _ = CASES[case]
    reqs, ref, mixed_reqs, mixed_ref = expected[case]
    runner = make_runner(folders[case], dtype, page_size, pool_tokens=helpers.round64(max(lengths)))
    for trace, what in ((helpers.trace_whole(reqs), "whole"), (helpers.trace_last_decoded(reqs, 32), "last 32 decoded"),
                        (helpers.trace_portions(reqs, seed=2), "portions")):
        got = helpers.run_trace(runner, trace)
        helpers.assert_logits_close(got, ref, TOL[dtype], f"lefavik {case} {dtype} {what}")
        runner.cache.check_invariants()
        assert not runner.cache.requests
    runner.runtime.kernels.check_error_word()
    pool = 384
    trace = helpers.trace_mixed(mixed_reqs, pool, seed=6)
    assert sum(helpers.round64(len(v)) for v in mixed_reqs.values()) > pool       # pages and slots are used again
    runner2 = make_runner(folders[case], dtype, page_size, pool)
    got = helpers.run_trace(runner2, trace)
    helpers.assert_logits_close(got, mixed_ref, TOL[dtype], f"lefavik {case} {dtype} mixed")
    runner2.cache.check_invariants()
    assert not runner2.cache.requests


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_blocks_other_ways(folders, expected, dtype, monkeypatch):
    """The same model with one branch's product after the other, and with the branches summed in an array of their own."""
    from chibillm_b200.parts import attention, latent_attention, mlp
    reqs, ref = expected["L3"][:2]
    runner = make_runner(folders["L3"], dtype, 16, 320)
    for b in runner.model.blocks:
        b.direct = b.hold = b.scaled_ok = False
    helpers.assert_logits_close(helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 20)), ref, TOL[dtype],
                                f"lefavik L3 {dtype}, branches apart")
    for part in (attention.PagedAttention, latent_attention.LatentAttention, mlp.GatedMLP):
        monkeypatch.setattr(part, "can_hold", False)
    runner = make_runner(folders["L3"], dtype, 16, 320)
    helpers.assert_logits_close(helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 20)), ref, TOL[dtype],
                                f"lefavik L3 {dtype}, one branch after the other")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_against_each_request_alone(folders, dtype):
    """Four unequal requests in the same steps against each in steps of its own, both against the plain
    implementation."""
    cfg = lefavik_models.get("L3")
    reqs = helpers.random_requests(cfg["vocab"], [90, 7, 140, 33], seed=17)
    ref = lefavik_models.plain_logits(cfg, SEED, reqs)
    runner = make_runner(folders["L3"], dtype, 16, 512)
    alone = helpers.run_trace(runner, helpers.trace_portions(reqs, seed=3))
    helpers.assert_logits_close(alone, ref, TOL[dtype], f"lefavik L3 {dtype} each alone")
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
    helpers.assert_logits_close(together, ref, TOL[dtype], f"lefavik L3 {dtype} together")
    helpers.assert_logits_close(together, alone, TOL[dtype], f"lefavik L3 {dtype} together against alone")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_long_prompt_whole_and_in_portions(folders, dtype):
    """1,500 tokens through the model of tensor-core sizes: whole, in portions of about 100 tokens and with its
    last 40 tokens decoded."""
    cfg = lefavik_models.get("L3")
    reqs = helpers.random_requests(cfg["vocab"], [1500], seed=31)
    ref = lefavik_models.plain_logits(cfg, SEED, reqs)
    runner = make_runner(folders["L3"], dtype, 16, 1536)
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
        helpers.assert_logits_close(helpers.run_trace(runner, trace), ref, TOL[dtype], f"lefavik L3 {dtype} long prompt {what}")
    runner.runtime.kernels.check_error_word()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(folders, dtype):
    """Three tokens of prompt, then 300 tokens one by one (captured steps replayed) across pages and windows."""
    cfg = lefavik_models.get("L1")
    reqs = helpers.random_requests(cfg["vocab"], [303], seed=9)
    ref = lefavik_models.plain_logits(cfg, SEED, reqs)
    runner = make_runner(folders["L1"], dtype, 4, 320)
    got = helpers.run_trace(runner, helpers.trace_last_decoded(reqs, 300))
    helpers.assert_logits_close(got, ref, TOL[dtype], f"lefavik L1 {dtype} long decoding")
    assert runner.graph_replays > 200


def test_greedy_generation_through_the_entry_point(folders):
    """``LLM.generate`` (scheduler, sampler, portions of 16 tokens, three requests at a time): every generated
    token is the plain implementation's best one, wherever that leads by more than the rounding of a 32-bit
    run."""
    from chibillm_b200 import LLM
    cfg = lefavik_models.get("L3")
    prompts = list(helpers.random_requests(cfg["vocab"], [5, 40, 23, 61], seed=12).values())
    llm = LLM(folders["L3"], dtype="float32", context_length=128, max_sequences=3, max_batch_tokens=48,
              prefill_chunk_tokens=16, page_size=16)
    outs = llm.generate(prompts, max_tokens=12, ignore_eos=True)
    for prompt, new in zip(prompts, outs):
        assert len(new) == 12
        ref = lefavik_models.plain_logits(cfg, SEED, {"a": prompt + new})["a"]
        for i, tok in enumerate(new):
            row = ref[len(prompt) + i - 1]
            top = torch.topk(row, 2).values
            if float(top[0] - top[1]) > 1e-3 * float(row.abs().max()):
                assert int(torch.argmax(row)) == tok, f"token {i} of a prompt of {len(prompt)}"


def test_trace_program(folders, tmp_path):
    """bin/trace_run on a Lefavik folder: portions, single tokens, two live requests."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = lefavik_models.get("L4")
    reqs = helpers.random_requests(cfg["vocab"], [40, 21], seed=5)
    ref = lefavik_models.plain_logits(cfg, SEED, reqs)
    a, b = reqs["r0"], reqs["r1"]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": [0]},
                                     {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[19:], "want": [0, 1]},
                                     {"id": "a", "tokens": a[31:], "want": [8]}], "end": ["a", "b"]}]
    want = [[("r0", 0), ("r0", 29)], [("r0", 30), ("r1", 18)], [("r1", 19), ("r1", 20), ("r0", 39)]]
    for dtype in ("float32", "bfloat16"):
        out_dir = str(tmp_path / dtype)
        proc = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["L4"], "--dtype",
                               dtype, "--out", out_dir, "--max-tokens", "128"],
                              input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True,
                              timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        for i, rows in enumerate(want):
            got = torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{i}.f32"), dtype="<f4").reshape(len(rows), -1))
            for j, (r, pos) in enumerate(rows):
                scale = float(ref[r].abs().max())
                assert float((got[j] - ref[r][pos]).abs().max()) <= TOL[dtype] * scale, (dtype, i, r, pos)


def test_random_weights_made_on_the_device(tmp_path):
    """``ModelRunner.from_random`` makes on the device the values that ``write_random_model`` stores: both
    give the same logits."""
    from chibillm_b200.engine.batch import StepEntry
    from chibillm_b200.engine.runner import ModelRunner
    from chibillm_b200.weights import write_random_model
    cfg = lefavik_models.get("L4")
    folder = write_random_model(cfg, str(tmp_path / "random"), seed=6)
    ids = helpers.random_requests(cfg["vocab"], [50], seed=2)["r0"]
    a = ModelRunner.from_folder(folder, dtype="float32", device=DEV, page_size=8, pool_tokens=64)
    b = ModelRunner.from_random(cfg, seed=6, dtype="float32", device=DEV, page_size=8, pool_tokens=64)
    la = a.step([StepEntry("x", ids, list(range(50)))]).clone()
    lb = b.step([StepEntry("x", ids, list(range(50)))]).clone()
    assert torch.equal(la, lb)
