"""Megerax on the GPU: every new kernel alone against plain float64 formulas, then the whole model through the
engine (prompts whole, in portions, token by token, in unequal batches, with slots and pages used again, long
decoding, greedy generation, trace replay, the command line) against tests/plain_megerax.py."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

import plain_megerax as P
from megerax_tiny import MG_CONFIGS, folder_config, make_megerax_folder, random_config
from test_gpu_birepel import argmax_lowest, paged
from test_gpu_loduzen import DTYPES, ROOT, TOL, TORCH, Tally, back, dev, engine, rel, step_tables
from tiny import random_prompts, read_weights

pytestmark = pytest.mark.gpu
D = torch.float64


@pytest.fixture(scope="module")
def K():
    from braidinfer_b200.csrc.api import get_kernels
    return get_kernels(verbose=False)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("megerax")
    return {n: make_megerax_folder(base, n) for n in MG_CONFIGS}


class Oracle:
    def __init__(self, folder):
        self.cfg, self.w, self.memo = folder_config(folder), read_weights(folder), {}

    def logits(self, tokens):
        key = tuple(tokens)
        if key not in self.memo:
            self.memo[key] = P.forward(self.cfg, self.w, list(tokens))
        return self.memo[key]


@pytest.fixture(scope="module")
def oracles(folders):
    return {n: Oracle(f) for n, f in folders.items()}


def tables_of(counts, before):
    return step_tables([n for n in counts if n], [b for n, b in zip(counts, before) if n], [i for i, n in enumerate(counts) if n], pad=1)


# ================================================================== kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nqh, nkh, dk, dv, taps, rot, adjacent, biased, normed", [
    (4, 2, 32, 48, 4, 16, True, True, True), (3, 3, 40, 20, 5, 0, True, True, True), (2, 1, 64, 64, 2, 64, True, False, True),
    (2, 2, 24, 8, 3, 20, True, True, False), (3, 1, 18, 12, 4, 8, False, True, True), (2, 1, 256, 136, 4, 32, True, True, True),
    (2, 2, 16, 16, 1, 16, True, True, True), (1, 1, 128, 32, 4, 128, False, False, True), (5, 0, 48, 0, 4, 24, True, True, True)])
def test_convolved_normed_rotated_heads_and_their_places_in_the_cache(K, dtype, nqh, nkh, dk, dv, taps, rot, adjacent, biased, normed):
    """Two sequences in portions (one of them across a page border), the inputs of earlier steps in their slots; `nkh` 0: a
    layer that reads another's keys and values."""
    g = torch.Generator().manual_seed(dk + dv + taps)
    page, eps, hd = 64, 1e-5, -(-max(dk, dv) // 16) * 16
    ch = nqh * dk + nkh * (dk + dv)
    lens = [70, 9]
    xs = [dev(torch.randn(n, ch, generator=g), dtype) for n in lens]
    b = dev(torch.randn(ch, generator=g), dtype) if biased else None
    w = dev(torch.randn(ch, taps, generator=g) * 0.5, dtype)
    qw, kw = (dev(1 + 0.3 * torch.randn(dk, generator=g), dtype) for _ in range(2)) if normed else (None, None)
    r = {"base": 500.0, "dims": rot}
    inv = P.frequencies(r).float().cuda()
    want = []
    for x in xs:
        y = P.causal_conv(back(x) + (back(b) if biased else 0.0), back(w))
        n = x.shape[0]
        pos = torch.arange(n)
        q = y[:, :nqh * dk].view(n, nqh, dk)
        k = y[:, nqh * dk:(nqh + nkh) * dk].view(n, nkh, dk)
        if normed:
            q, k = P.norm(q, back(qw), eps), P.norm(k, back(kw), eps)
        lay = "pairs" if adjacent else "half"
        want.append((P.rotate(q, pos, r, lay), P.rotate(k, pos, r, lay), y[:, (nqh + nkh) * dk:].view(n, nkh, dv)))
    tol = 1e-5 if dtype == "float32" else 1e-2
    for cuts in ([[70, 9]], [[1, 1], [2, 2], [61, 1], [6, 5]], [[20, 0], [1, 3], [49, 6]], [[1, 1]] * 9 + [[61, 0]]):
        table, cache = paged(lens, max(nkh, 1), page, hd, dtype, g)
        state = torch.zeros(3, max((taps - 1) * ch * 4, 16), dtype=torch.uint8, device="cuda")
        before = [0, 0]
        for counts in cuts:
            t = tables_of(counts, before)
            rows = torch.cat([xs[i][before[i]:before[i] + n] for i, n in enumerate(counts)] + [torch.full((1, ch), 9.0, dtype=TORCH[dtype], device="cuda")])
            wide = torch.cat([rows, torch.full((rows.shape[0], 8), 5.0, dtype=TORCH[dtype], device="cuda")], 1)     # a view, as the mixer passes it
            q_out = torch.full((t.rows, nqh * hd), 3.0, dtype=TORCH[dtype], device="cuda")
            segs = [K.conv_segment(nqh, dk, pad=hd, norm="rms" if normed else None, weight=qw, rotate=True, out=q_out)]
            if nkh:
                segs += [K.conv_segment(nkh, dk, pad=hd, norm="rms" if normed else None, weight=kw, rotate=True, plane=0),
                         K.conv_segment(nkh, dv, pad=hd, plane=1)]
            live = [i for i, n in enumerate(counts) if n]
            K.conv_heads(wide[:, :ch], w, b, state, 0, t, segs, eps=eps, inv_freq=inv, adjacent=adjacent,
                         page_table=table[live].contiguous().cuda() if nkh else None, cache=cache if nkh else None)
            K.check_device_errors()
            r0 = 0
            for i in live:
                got = back(q_out)[r0:r0 + counts[i]].view(-1, nqh, hd)
                assert rel(got[..., :dk], want[i][0][before[i]:before[i] + counts[i]]) < tol and got[..., dk:].abs().sum().item() == 0, (cuts, counts)
                r0 += counts[i]
                before[i] += counts[i]
            assert (q_out[r0:] == 3.0).all()                                  # the padding row is left alone
        for i in range(2):
            for j in range(lens[i] if nkh else 0):
                pg = int(table[i, j // page])
                kk, vv = back(cache[pg, 0, :, j % page]), back(cache[pg, 1, :, j % page])
                assert rel(kk[:, :dk], want[i][1][j]) < tol and rel(vv[:, :dv], want[i][2][j]) < tol, (cuts, i, j)
                assert kk[:, dk:].abs().sum().item() == 0 and vv[:, dv:].abs().sum().item() == 0
            if taps > 1:                                                       # the state holds the last inputs, bias and all
                st = state[i].view(torch.float32)[:(taps - 1) * ch].view(taps - 1, ch)
                assert torch.allclose(st.cpu(), (xs[i].float() + (b.float() if biased else 0.0))[-(taps - 1):].cpu(), atol=1e-6)
        used = sum(lens)
        assert nkh == 0 or int((cache.abs().amax((1, 2, 4)) > 0).sum()) == used


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dk, dv, taps", [(4, 2, 24, 40, 3), (3, 3, 128, 64, 4), (2, 1, 33, 7, 4), (2, 2, 8, 8, 1)])
def test_convolution_with_silu_and_unit_heads_in_32_bits(K, dtype, H, G, dk, dv, taps):
    g = torch.Generator().manual_seed(dk)
    ch, n = 2 * G * dk + H * dv, 37
    x, w = dev(torch.randn(n, ch, generator=g), dtype), dev(torch.randn(ch, taps, generator=g), dtype)
    state = torch.zeros(2, max((taps - 1) * ch * 4, 16), dtype=torch.uint8, device="cuda")
    y = P.silu(P.causal_conv(back(x), back(w)))
    want = [P.unit_heads(y[:, :G * dk].view(n, G, dk)) * dk ** -0.5, P.unit_heads(y[:, G * dk:2 * G * dk].view(n, G, dk)), y[:, 2 * G * dk:].view(n, H, dv)]
    got = [[], [], []]
    for a, b in ((0, 5), (5, 6), (6, 8), (8, 37)):
        t = step_tables([b - a], [a])
        outs = [torch.zeros(b - a, m, dtype=torch.float32, device="cuda") for m in (G * dk, G * dk, H * dv)]
        K.conv_heads(x[a:b], w, None, state, 0, t, [K.conv_segment(G, dk, silu=True, norm="unit", factor=dk ** -0.5, out=outs[0]),
                                                   K.conv_segment(G, dk, silu=True, norm="unit", out=outs[1]),
                                                   K.conv_segment(H, dv, silu=True, out=outs[2])], eps=1e-6)
        for gg, o in zip(got, outs):
            gg.append(o)
    for gg, o in zip(got, want):
        assert rel(torch.cat(gg).view(o.shape), o) < 3e-6                       # nothing is rounded to 16 bits on the way
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nqh, nkh, hd, taps, rot", [(3, 1, 16, 4, 8), (4, 2, 64, 3, 64), (2, 2, 128, 2, 32), (5, 1, 48, 4, 16)])
def test_convolved_heads_of_many_rows_and_sequences(K, dtype, nqh, nkh, hd, taps, rot):
    """Steps of so many rows that a CTA walks a span of them: long sequences, short ones that begin and end anywhere in a span,
    hundreds of one token, over three steps with the inputs between them in the slots; rows of padding in the middle of nothing."""
    g = torch.Generator().manual_seed(hd)
    page, eps, ch = 64, 1e-5, (nqh + 2 * nkh) * hd
    first = [2111, 1, 2, 5, 700, 3] + [1] * 300
    steps = [first, [40, 1, 7, 1, 1500, 2] + [1] * 900, [1] * 2600]
    n_seqs = max(len(c) for c in steps)
    total = [sum(c[i] for c in steps if i < len(c)) for i in range(n_seqs)]
    xs = [dev(torch.randn(n, ch, generator=g), dtype) for n in total]
    b, w = dev(torch.randn(ch, generator=g), dtype), dev(torch.randn(ch, taps, generator=g) * 0.5, dtype)
    qw, kw = (dev(1 + 0.3 * torch.randn(hd, generator=g), dtype) for _ in range(2))
    r = {"base": 500.0, "dims": rot}
    inv = P.frequencies(r).float().cuda()
    # the plain result, all sequences as one batch with zeros before each start
    flat = torch.cat([torch.cat([torch.zeros(taps - 1, ch, dtype=D), back(x) + back(b)]) for x in xs])
    y = P.causal_conv(flat, back(w))
    keep = torch.cat([torch.arange(n) + taps - 1 + at for n, at in zip(total, torch.tensor([0] + [n + taps - 1 for n in total[:-1]]).cumsum(0).tolist())])
    y, pos = y[keep], torch.cat([torch.arange(n) for n in total])
    starts = torch.tensor([0] + total[:-1]).cumsum(0).tolist()
    q = P.rotate(P.norm(y[:, :nqh * hd].view(-1, nqh, hd), back(qw), eps), pos, r, "pairs")
    k = P.rotate(P.norm(y[:, nqh * hd:(nqh + nkh) * hd].view(-1, nkh, hd), back(kw), eps), pos, r, "pairs")
    v = y[:, (nqh + nkh) * hd:].view(-1, nkh, hd)
    table, cache = paged(total, nkh, page, hd, dtype, g)
    state, at = torch.zeros(n_seqs, (taps - 1) * ch * 4, dtype=torch.uint8, device="cuda"), [0] * n_seqs
    tol = 3e-4 if dtype == "float32" else 1.2e-2                                # (angles of thousands of radians in float32)
    for counts in steps:
        m = len(counts)
        t = step_tables(counts, at[:m], pad=3)
        rows = torch.cat([xs[i][at[i]:at[i] + n] for i, n in enumerate(counts)] + [torch.full((3, ch), 9.0, dtype=TORCH[dtype], device="cuda")])
        q_out = torch.full((t.rows, nqh * hd), 3.0, dtype=TORCH[dtype], device="cuda")
        head = dict(norm="rms", rotate=True)
        K.conv_heads(rows, w, b, state, 0, t, [K.conv_segment(nqh, hd, weight=qw, out=q_out, **head), K.conv_segment(nkh, hd, weight=kw, plane=0, **head),
                                              K.conv_segment(nkh, hd, plane=1)], eps=eps, inv_freq=inv, page_table=table[:m].contiguous().cuda(), cache=cache)
        K.check_device_errors()
        where = torch.cat([torch.arange(at[i], at[i] + n) + starts[i] for i, n in enumerate(counts)])
        assert rel(q_out[:t.n_tokens], q[where].reshape(len(where), -1)) < tol and (q_out[t.n_tokens:] == 3.0).all()
        at = [x + (counts[i] if i < m else 0) for i, x in enumerate(at)]
    seq = torch.repeat_interleave(torch.arange(n_seqs), torch.tensor(total))
    pg = table[seq, pos // page].long().cuda()
    assert rel(cache[pg, 0, :, (pos % page).cuda()], k) < tol and rel(cache[pg, 1, :, (pos % page).cuda()], v) < (1e-5 if dtype == "float32" else 1e-2)
    for i in (0, 1, 2, 4, 5, 200, 1100, 2599):
        u = torch.cat([torch.zeros(taps - 1, ch), xs[i].float().cpu() + b.float().cpu()])[-(taps - 1):]
        assert torch.allclose(state[i].view(torch.float32).view(taps - 1, ch).cpu(), u, atol=1e-6)
    # the delta layer's form on the same rows: silu, unit heads, float32 results, values in heads twice as wide
    t = step_tables(first, [0] * len(first))
    rows = torch.cat([xs[i][:n] for i, n in enumerate(first)])
    wide = nqh + 2 * nkh
    G, rest = (wide // 4, wide - 2 * (wide // 4)) if wide >= 4 else (1, wide - 2)
    if rest % 2:
        return
    outs = [torch.zeros(t.rows, n, dtype=torch.float32, device="cuda") for n in (G * hd, G * hd, rest * hd)]
    st2 = torch.zeros(len(first), (taps - 1) * ch * 4, dtype=torch.uint8, device="cuda")
    K.conv_heads(rows, w, None, st2, 0, t, [K.conv_segment(G, hd, silu=True, norm="unit", factor=0.25, out=outs[0]),
                                            K.conv_segment(G, hd, silu=True, norm="unit", out=outs[1]),
                                            K.conv_segment(rest // 2, 2 * hd, silu=True, out=outs[2])], eps=1e-6)
    r0 = 0
    for i, n in enumerate(first[:30]):
        z = P.silu(P.causal_conv(back(xs[i][:n]), back(w)))
        assert rel(outs[0][r0:r0 + n], (P.unit_heads(z[:, :G * hd].view(n, G, hd)) * 0.25).reshape(n, -1)) < 5e-6
        assert rel(outs[1][r0:r0 + n], P.unit_heads(z[:, G * hd:2 * G * hd].view(n, G, hd)).reshape(n, -1)) < 5e-6
        assert rel(outs[2][r0:r0 + n], z[:, 2 * G * hd:]) < 5e-6
        r0 += n


def delta_inputs(g, n, H, G, dk, dv, dtype, spread=2.0, shift=-4.0):
    unit = lambda x: x / x.norm(dim=-1, keepdim=True)                           # noqa: E731
    q, k = (unit(torch.randn(n, G, dk, generator=g)) for _ in range(2))
    return [q, k, torch.randn(n, H, dv, generator=g), torch.randn(n, H, dk, generator=g) * spread + shift,
            dev(torch.randn(n, H, generator=g) * 2, dtype)]


def plain_delta(seq, bias, rate, H, G, S=None):
    q, k, v, z, b = (back(x) for x in seq)
    of = torch.arange(H) // (H // G)
    decay = torch.exp(-rate.double()[None, :, None] * P.softplus(z + bias.double().view(1, H, -1)))
    return P.delta_rule(q[:, of], k[:, of], v, decay, P.sigmoid(b), S)


def run_delta(K, seqs, slices, slots, state, bias, rate, H, G, dk, dv, chunked, offset=0):
    """One step: sequence i brings seqs[i][slices[i]]."""
    lens = [s.stop - s.start for s in slices]
    live = [i for i, n in enumerate(lens) if n]
    t = step_tables([lens[i] for i in live], [slices[i].start for i in live], [slots[i] for i in live], pad=2)
    cat = lambda j, m: torch.cat([seqs[i][j][slices[i]].reshape(lens[i], -1).cuda() for i in live]       # noqa: E731
                                 + [torch.full((2, m), 1e4, dtype=seqs[0][j].dtype, device="cuda")])
    out = torch.full((t.rows, H * dv), 3.0, dtype=torch.float32, device="cuda")
    K.delta_rule(cat(0, G * dk), cat(1, G * dk), cat(2, H * dv), cat(3, H * dk), bias.cuda(), rate.cuda(), cat(4, H), out, state, offset, t,
                 H, G, dk, dv, chunked)
    torch.cuda.synchronize()
    K.check_device_errors()
    assert (out[t.n_tokens:] == 3.0).all()
    res, r0 = {}, 0
    for i in live:
        res[i] = back(out[r0:r0 + lens[i]]).view(-1, H, dv)
        r0 += lens[i]
    return res


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, G, dk, dv", [(4, 2, 24, 40), (3, 1, 136, 36), (2, 2, 33, 70), (8, 4, 8, 8), (2, 1, 128, 128), (1, 1, 64, 4),
                                          (2, 2, 200, 33), (6, 3, 32, 130), (1, 1, 1, 1)])
def test_delta_rule_token_by_token_in_portions_and_over_chunks(K, dtype, H, G, dk, dv):
    g = torch.Generator().manual_seed(dk + dv)
    lens = [201, 77, 15]
    seqs = [delta_inputs(g, n, H, G, dk, dv, dtype) for n in lens]
    bias, rate = torch.randn(H * dk, generator=g), torch.rand(H, generator=g) * 2 + 0.1
    want = [plain_delta(s, bias, rate, H, G) for s in seqs]
    off = 48                                                                    # the matrix does not start the slot
    cuts = [([201, 77, 15], True), ([201, 77, 15], False), [([64, 64, 0], True), ([63, 13, 15], True), ([74, 0, 0], True)],
            [([2, 0, 3], False), ([1, 1, 1], False), ([130, 60, 11], True), ([68, 16, 0], False)], [([65, 1, 1], True)] * 3 + [([6, 74, 12], True)]]
    for plan in cuts:
        state = torch.zeros(5, off + H * dk * dv * 4, dtype=torch.uint8, device="cuda")
        at, got = [0, 0, 0], [[], [], []]
        for counts, chunked in (plan if isinstance(plan, list) else [plan]):
            sl = [slice(a, a + c) for a, c in zip(at, counts)]
            for i, o in run_delta(K, seqs, sl, [3, 0, 2], state, bias, rate, H, G, dk, dv, chunked, off).items():
                got[i].append(o)
            at = [s.stop for s in sl]
        for i in range(3):
            S = back(state[[3, 0, 2][i], off:].view(torch.float32)).view(H, dk, dv)
            assert rel(torch.cat(got[i]), want[i][0]) < 1e-5 and rel(S, want[i][1]) < 1e-5, (plan, i)
        assert state[1].abs().max() == 0 and state[4].abs().max() == 0


def test_delta_rule_over_chunks_of_many_sequences_of_unequal_lengths(K):
    """Chunks are packed one after the other: sequences that end anywhere, some of one token, in two steps."""
    g = torch.Generator().manual_seed(8)
    H, G, dk, dv = 2, 1, 20, 18
    lens = [1, 64, 65, 130, 63, 2, 128, 1, 127, 200, 3, 61]
    seqs = [delta_inputs(g, n, H, G, dk, dv, "float32") for n in lens]
    bias, rate = torch.randn(H * dk, generator=g), torch.rand(H, generator=g) + 0.1
    state = torch.zeros(len(lens), H * dk * dv * 4, dtype=torch.uint8, device="cuda")
    cut = [(n + 1) // 2 for n in lens]
    a = run_delta(K, seqs, [slice(0, c) for c in cut], list(range(len(lens))), state, bias, rate, H, G, dk, dv, True)
    b = run_delta(K, seqs, [slice(c, n) for c, n in zip(cut, lens)], list(range(len(lens))), state, bias, rate, H, G, dk, dv, True)
    for i, s in enumerate(seqs):
        want, S = plain_delta(s, bias, rate, H, G)
        assert rel(torch.cat([a[i]] + ([b[i]] if i in b else [])), want) < 1e-5, i
        assert rel(back(state[i].view(torch.float32)).view(H, dk, dv), S) < 1e-5, i


@pytest.mark.parametrize("dk", [32, 64, 128, 256])
def test_delta_rule_over_chunks_with_channels_that_forget_at_once(K, dk):
    """Some channels lose everything at a token (decays down to exp(-1000)), others keep nearly everything: no overflow, and the
    slow ones keep their precision.  A sub-chunk with a steep channel takes another way through the kernel than one without."""
    g = torch.Generator().manual_seed(dk)
    H, G, dv, n = 2, 1, 20, 150
    seq = delta_inputs(g, n, H, G, dk, dv, "float32", spread=0.5, shift=-6.0)
    seq[3][torch.rand(n, H, dk, generator=g) < 0.02] = 1000.0
    seq[3][70:75, :, :dk // 2] = 30.0
    seq[3][20:64, 1] = 5.0                                                      # a head steep all along
    bias, rate = torch.zeros(H * dk), torch.tensor([1.0, 3.0])
    want, S = plain_delta(seq, bias, rate, H, G)
    for chunked in (True, False):
        state = torch.zeros(1, H * dk * dv * 4, dtype=torch.uint8, device="cuda")
        got = run_delta(K, [seq], [slice(0, n)], [0], state, bias, rate, H, G, dk, dv, chunked)[0]
        assert torch.isfinite(got).all() and rel(got, want) < 1e-5, chunked
        assert rel(back(state[0].view(torch.float32)).view(H, dk, dv), S) < 1e-5, chunked


@pytest.mark.parametrize("chunked", [True, False])
def test_delta_rule_reads_a_write_from_a_thousand_tokens_back(K, chunked):
    """The first token writes at a key that no later token comes near; every 100th token reads at it.  Half of the channels
    decay slowly, by a known factor, and beta is one."""
    H = G = 1
    dk, dv, n = 64, 16, 1100
    g = torch.Generator().manual_seed(3)
    k = torch.zeros(n, 1, dk)
    k[:, 0, 1:] = torch.randn(n, dk - 1, generator=g)
    k /= k.norm(dim=-1, keepdim=True)
    k[0] = torch.eye(dk)[0]
    q = k.roll(1, 0).clone()
    q[::100, 0] = torch.eye(dk)[0]
    z = torch.full((n, 1, dk), math.log(math.expm1(0.001)))                     # softplus(z) = 0.001
    v = torch.randn(n, 1, dv, generator=g)
    v[0] = 40.0
    seq = [q, k, v, z, torch.full((n, 1), 30.0)]
    bias, rate = torch.zeros(dk), torch.ones(1)
    want, _ = plain_delta(seq, bias, rate, H, G)
    assert abs(want[1000, 0, 0].item() - 40.0 * math.exp(-1.0)) < 1e-3
    state = torch.zeros(1, dk * dv * 4, dtype=torch.uint8, device="cuda")
    got = torch.cat([run_delta(K, [seq], [slice(a, b)], [0], state, bias, rate, H, G, dk, dv, chunked)[0] for a, b in ((0, 333), (333, 1000), (1000, n))])
    # a thousand products with one rounded decay: its rounding counts a thousand times
    assert rel(got, want) < 6e-5 and (got[::100] - want[::100]).abs().max().item() < 3e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H, dv", [(3, 40), (2, 128), (5, 7), (2, 256), (1, 130)])
def test_read_out_norm_with_a_sigmoid_gate_in_32_bits(K, dtype, H, dv):
    g = torch.Generator().manual_seed(dv)
    y, gate = torch.randn(9, H * dv, generator=g).cuda(), torch.randn(9, H * dv + 4, generator=g).cuda()[:, 4:]
    w, out = dev(1 + 0.3 * torch.randn(dv, generator=g), dtype), torch.full((9, H * dv), 3.0, dtype=TORCH[dtype], device="cuda")
    seq = torch.tensor([0] * 8 + [-1], dtype=torch.int32, device="cuda")
    K.delta_gated_norm(y, gate, w, out, seq, dv, 1e-5)
    want = (P.norm(back(y).view(9, H, dv), back(w), 1e-5).view(9, -1) * P.sigmoid(back(gate)))
    assert rel(out[:8], want[:8]) < (1e-6 if dtype == "float32" else 1e-2) and (out[8] == 3.0).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, hd, dv", [(3, 48, 40), (2, 48, 20), (1, 16, 16), (4, 128, 32), (3, 16, 5)])
def test_a_gate_a_column_on_the_heads(K, dtype, heads, hd, dv):
    g = torch.Generator().manual_seed(hd + dv)
    x, gate = dev(torch.randn(7, heads * hd, generator=g), dtype), dev(torch.randn(7, heads * dv + 8, generator=g) * 3, dtype)[:, 8:]
    out = torch.empty(7, heads * dv, dtype=TORCH[dtype], device="cuda")
    K.head_gate(x, gate, out, heads, hd, dv, per_column=True)
    want = back(x).view(7, heads, hd)[..., :dv].reshape(7, -1) * P.sigmoid(back(gate))
    assert rel(out, want) < (1e-6 if dtype == "float32" else 1e-2)
    K.head_gate(x, None, out, heads, hd, dv)
    assert torch.equal(back(out), back(x).view(7, heads, hd)[..., :dv].reshape(7, -1))


def plain_capped(q, keys, vals, positions, scale, cap, nkh, size):
    """q [n, H, hd]; keys, vals [T, nkh, hd]; float64."""
    n, H, hd = q.shape
    j = torch.arange(keys.shape[0])
    d = positions[:, None] - j[None, :]
    vis = (d >= 0) & (d < size)
    out = torch.zeros(n, H, hd, dtype=D)
    for a in range(H):
        c = a // (H // nkh)
        out[:, a] = P.masked_softmax(P.capped((q[:, a] @ keys[:, c].T) * scale, cap)[None], vis[None])[0] @ vals[:, c]
    return out


@pytest.mark.parametrize("kernel", ["simple_f32", "simple_bf16", "mma_prompt", "mma_few_1", "mma_few_7", "tcgen05_prompt"])
@pytest.mark.parametrize("nqh, nkh, hd, size, cap", [(4, 2, 48, 40, 5.0), (6, 3, 16, 64, 20.0), (3, 3, 48, 7, 8.0), (8, 1, 64, 70, 6.0),
                                                     (4, 4, 128, 96, 12.0), (2, 1, 64, 300, 50.0), (2, 2, 32, 1, 5.0), (4, 1, 128, 65, 4.0),
                                                     (6, 2, 64, 127, 9.0), (5, 1, 96, 1000, 100.0)])
def test_attention_with_capped_scores_behind_a_window(K, kernel, nqh, nkh, hd, size, cap):
    """For the last query of each sequence three keys stand out alike, with large values: the oldest one inside the window, the one
    just outside, and the query's own; their scores lie far beyond the cap, the others' well below it.  The cap a little larger or
    a score left as it was would show."""
    if kernel == "tcgen05_prompt" and hd not in (64, 128):
        pytest.skip("the tcgen05 kernel takes heads of 64 and 128")
    g = torch.Generator().manual_seed(nqh * hd + size)
    dtype = "float32" if kernel == "simple_f32" else "bfloat16"
    few = kernel.startswith("mma_few")
    n_few = int(kernel[-1]) if few else 0
    lengths, before = ([n_few, 1], [320 - n_few, 131]) if few else ([150, 37], [0, 290])
    t = step_tables(lengths, before, pad=1)
    total = [b + n for b, n in zip(before, lengths)]
    page, scale = 64, 2.0 / math.sqrt(hd)
    table, cache = paged(total, nkh, page, hd, dtype, g)
    keys, vals = [torch.randn(n, nkh, hd, generator=g) for n in total], [torch.randn(n, nkh, hd, generator=g) for n in total]
    u = torch.ones(hd) / math.sqrt(hd)
    for s in range(2):
        for j in {total[s] - 1 - size, total[s] - size, total[s] - 1}:
            if j >= 0:
                keys[s][j] = 1.5 * cap * u / (4.0 * scale)                     # with the queries' lean: a score of about 1.5 cap
                vals[s][j] = 5.0 * torch.sign(torch.randn(nkh, hd, generator=g))
        for j in range(total[s]):
            pg = int(table[s, j // page])
            cache[pg, 0, :, j % page] = dev(keys[s][j], dtype)
            cache[pg, 1, :, j % page] = dev(vals[s][j], dtype)
    q0 = torch.randn(t.rows, nqh * hd + 8, generator=g)
    q0[:, :nqh * hd] += (4.0 * u).repeat(nqh)
    q = dev(q0, dtype)
    out = torch.full((t.rows, nqh * hd), 7.0, dtype=TORCH[dtype], device="cuda")
    if kernel.startswith("simple"):
        K.attn_simple(q, out, cache, table.cuda(), t.positions, t.token_seq, nqh, nkh, hd, page, size, scale, softcap=cap)
    elif kernel == "tcgen05_prompt":
        K.attn_tc(q, out, cache, table.cuda(), t.q_start, t.q_len, t.kv_before, 2, max(lengths), nqh, nkh, hd, size, scale, softcap=cap)
    else:
        K.attn_mma(q, out, cache, table.cuda(), t.q_start, t.q_len, t.kv_before, t.token_seq, t.n_seqs, t.max_q_len, nqh, nkh, hd, size,
                   scale, n_splits=1 if not few else 3 if size > 128 else 2, few_tokens=few, softcap=cap)
    K.check_device_errors()
    qs, r0, shown = back(q)[:, :nqh * hd].view(-1, nqh, hd), 0, [0.0, 0.0, 0.0]
    for s in range(2):
        rows = slice(r0, r0 + lengths[s])
        pos = torch.arange(before[s], total[s])
        kk, vv = back(dev(keys[s], dtype)), back(dev(vals[s], dtype))
        want = plain_capped(qs[rows], kk, vv, pos, scale, cap, nkh, size)
        assert rel(back(out)[rows].view(-1, nqh, hd), want) < (2e-5 if dtype == "float32" else 3e-2), (kernel, s)
        for i, (c2, sz) in enumerate(((cap, size + 1), (cap, max(size - 1, 1)), (1.5 * cap, size))):       # what faults would give
            shown[i] = max(shown[i], rel(plain_capped(qs[rows], kk, vv, pos, scale, c2, nkh, sz), want))
        r0 += lengths[s]
    if size < min(total):
        assert shown[0] > 0.15 and (size == 1 or shown[1] > 0.15)               # the test's inputs do show a window off by one
    assert size < 64 or cap > 10 or shown[2] > 0.05                             # and another cap, where many scores are near it


def test_capped_scores_are_exact_from_small_to_far_beyond_the_cap(K):
    """Both forms of the tanh: with one key and a sink-like second key of score 0 the result is sigmoid(capped score)."""
    hd, page, cap, scale = 64, 64, 10.0, 1.0
    want_scores = torch.tensor([-300.0, -40.0, -9.0, -7.6, -7.4, -3.0, -0.5, -1e-3, 0.0, 1e-3, 0.3, 2.0, 7.45, 7.55, 8.0, 15.0, 60.0, 500.0], dtype=D)
    n = len(want_scores)
    cache = torch.zeros(1, 2, 1, page, hd, dtype=torch.float32, device="cuda")
    cache[0, 0, 0, 1, 0] = 1.0                                                   # key 1: reads the query's first number; key 0: nothing
    cache[0, 1, 0, 1, :] = 1.0
    for one in range(2):
        for dtype in DTYPES:
            c = cache.to(TORCH[dtype])
            q = torch.zeros(n, hd, dtype=TORCH[dtype], device="cuda")
            q[:, 0] = want_scores.to(TORCH[dtype]).cuda()
            real = back(q)[:, 0]
            w = P.sigmoid(cap * torch.tanh(real / cap))
            table = torch.zeros(n, 1, dtype=torch.int32, device="cuda")
            i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")    # noqa: E731
            out = torch.zeros(n, hd, dtype=TORCH[dtype], device="cuda")
            if dtype == "float32":
                K.attn_simple(q, out, c, table, i32([1] * n), i32(list(range(n))), 1, 1, hd, page, None, scale, softcap=cap)
            elif one:
                K.attn_mma(q, out, c, table, i32(list(range(n))), i32([1] * n), i32([1] * n), i32(list(range(n))), n, 1, 1, 1, hd, None, scale,
                           few_tokens=True, softcap=cap)
            else:
                K.attn_tc(q, out, c, table, i32(list(range(n))), i32([1] * n), i32([1] * n), n, 1, 1, 1, hd, None, scale, softcap=cap)
            assert ((back(out)[:, 5] - w).abs() / (w + 1e-4)).max().item() < (2e-6 if dtype == "float32" else 1e-2), (dtype, one)
    K.check_device_errors()


def plain_sink_latent(q, keys, positions, rank, scale, sinks):
    T = keys.shape[0]
    vis = torch.arange(T)[None, :] <= positions[:, None]
    s = torch.einsum("nhd,td->hnt", q, keys) * scale
    return torch.einsum("hnt,tr->nhr", P.masked_softmax(s, vis[None], sinks), keys[:, :rank])


@pytest.mark.parametrize("kernel", ["simple_f32", "simple_bf16", "mma_prompt", "mma_few", "mma_sliced", "mma_sliced_64"])
@pytest.mark.parametrize("rank, rot, heads", [(32, 16, 3), (64, 16, 4), (64, 16, 1), (16, 16, 7), (48, 16, 5)])
def test_latent_attention_with_a_sink_a_head(K, kernel, rank, rot, heads):
    """Sinks from far below to above every score; a sink counted once a slice, scaled, or left out moves the rows."""
    g = torch.Generator().manual_seed(rank + heads)
    dtype = "float32" if kernel == "simple_f32" else "bfloat16"
    lengths, before = {"mma_few": ([2, 1], [70, 200]), "mma_sliced": ([1, 1], [300, 200]), "mma_sliced_64": ([8, 8], [300, 133])}.get(kernel, ([130, 21], [0, 90]))
    if kernel == "mma_few" and heads > 6:
        pytest.skip("few pairs")
    t = step_tables(lengths, before, pad=1)
    total = [b + n for b, n in zip(before, lengths)]
    page, scale, Dl = 64, 0.3, rank + rot
    blocks = [-(-x // page) for x in total]
    perm = torch.randperm(sum(blocks) + 1, generator=g)
    table = torch.full((2, max(blocks)), -1, dtype=torch.int32)
    table[0, :blocks[0]], table[1, :blocks[1]] = perm[:blocks[0]].int(), perm[blocks[0]:blocks[0] + blocks[1]].int()
    cache = torch.zeros(sum(blocks) + 1, 1, 1, page, Dl, dtype=TORCH[dtype], device="cuda")
    keys = [dev(torch.randn(n, Dl, generator=g), dtype) for n in total]
    for s in range(2):
        for j in range(total[s]):
            cache[int(table[s, j // page]), 0, 0, j % page] = keys[s][j]
    q = dev(torch.randn(t.rows, heads, Dl, generator=g) * 0.6, dtype)
    sinks = torch.linspace(-30.0, 9.0, heads) if heads > 1 else torch.tensor([9.0])
    out = torch.full((t.rows, heads, rank), 7.0, dtype=TORCH[dtype], device="cuda")
    if kernel.startswith("simple"):
        K.attn_latent_simple(q, out, cache, table.cuda(), t.positions, t.token_seq, rank, None, scale, sinks=sinks.cuda())
    else:
        K.attn_latent_mma(q, out, cache, table.cuda(), t.q_start, t.q_len, t.kv_before, t.token_seq, t.n_seqs, t.max_q_len, rank, None, scale,
                          n_splits=3 if "sliced" in kernel else 1, sinks=sinks.cuda())
    K.check_device_errors()
    r0 = 0
    for s in range(2):
        pos, rows = torch.arange(before[s], total[s]), slice(r0, r0 + lengths[s])
        want = plain_sink_latent(back(q)[rows], back(keys[s]), pos, rank, scale, sinks.double())
        for h in range(heads):
            assert rel(back(out)[rows, h], want[:, h]) < (1e-5 if dtype == "float32" else 3e-2), (kernel, s, h)
        assert rel(plain_sink_latent(back(q)[rows], back(keys[s]), pos, rank, scale, torch.full((heads,), -1e9, dtype=D))[:, -1], want[:, -1]) > 0.2
        r0 += lengths[s]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank, rank, rot", [(40, 32, 16), (13, 20, 6), (64, 64, 16), (136, 80, 8), (7, 300, 2)])
def test_low_rank_queries_normed_beside_the_latent(K, dtype, q_rank, rank, rot):
    g = torch.Generator().manual_seed(q_rank)
    pad, page, eps = -(-q_rank // 8) * 8, 64, 1e-5
    lengths, before = [3, 70, 1], [0, 60, 129]
    t = step_tables(lengths, before, pad=1)
    proj = dev(torch.randn(t.rows, pad + rank + rot + 3, generator=g), dtype)
    wq, wc = dev(1 + 0.3 * torch.randn(q_rank, generator=g), dtype), dev(1 + 0.3 * torch.randn(rank, generator=g), dtype)
    r = {"base": 300.0, "dims": rot}
    table = torch.arange(9, dtype=torch.int32).view(3, 3)
    cache = torch.zeros(9, 1, 1, page, rank + rot, dtype=TORCH[dtype], device="cuda")
    c_q = torch.full((t.rows, pad), 5.0, dtype=TORCH[dtype], device="cuda")
    K.latent_down(proj, pad, c_q, wq, wc, P.frequencies(r).float().cuda(), t.positions, t.token_seq, table.cuda(), cache, rot, rank, rot, page, eps)
    K.check_device_errors()
    tol = 1e-5 if dtype == "float32" else 1e-2                                  # (angles are float32)
    p = back(proj)
    n = t.n_tokens
    assert rel(c_q[:n, :q_rank], P.norm(p[:n, :q_rank], back(wq), eps)) < tol and (c_q[:n, q_rank:] == 0).all()
    pos = t.positions.cpu()
    c, kr = P.norm(p[:, pad:pad + rank], back(wc), eps), P.rotate(p[:, None, pad + rank:pad + rank + rot], pos, r, "half")[:, 0]
    for row in range(n):
        s, j = int(t.token_seq[row]), int(pos[row])
        assert rel(cache[int(table[s, j // page]), 0, 0, j % page], torch.cat([c[row], kr[row]])) < tol
    assert int((cache.abs().amax(-1) > 0).sum()) == n


def test_kernels_refuse_what_does_not_fit(K):
    from braidinfer_b200.csrc.api import KernelError
    t = step_tables([2], [0])
    x, w, st = torch.zeros(2, 16, device="cuda"), torch.zeros(16, 3, device="cuda"), torch.zeros(1, 128, dtype=torch.uint8, device="cuda")
    o = torch.zeros(2, 16, device="cuda")
    for segs in ([K.conv_segment(1, 8, out=o)], [K.conv_segment(1, 16, pad=8, out=o)], [K.conv_segment(1, 16, norm="rms", out=o)], [K.conv_segment(1, 16)],
                 [K.conv_segment(2, 8, pad=16, out=o)], [K.conv_segment(1, 16, plane=2)]):
        with pytest.raises(KernelError):
            K.conv_heads(x, w, None, st, 0, t, segs, eps=1e-6)
    z = lambda *s: torch.zeros(*s, device="cuda")                               # noqa: E731
    with pytest.raises(KernelError):
        K.delta_rule(z(2, 300), z(2, 300), z(2, 4), z(2, 300), z(300), z(1), z(2, 1), z(2, 4), st, 0, t, 1, 1, 300, 4, False)
    with pytest.raises(KernelError):
        K.delta_rule(z(2, 8), z(2, 8), z(2, 4), z(2, 8), z(8), z(1), z(2, 1), z(2, 8), st, 0, t, 1, 1, 8, 4, False)
    with pytest.raises(KernelError):
        K.conv_segment(1, 1, norm="mean")


# ================================================================== the whole model through the engine
NAMES = ["A", "B", "C", "D"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_every_layer(folders, oracles, name, dtype):
    o = oracles[name]
    eng, tally = engine(folders[name], dtype), Tally(dtype)
    for n, seed in ((1, 0), (2, 1), (67, 2), (300, 3)):
        toks = random_prompts(o.cfg["vocab"], [n], seed)[0]
        s, taps = eng.open(), []
        got = eng.step([(s, toks)], want="all", tap=lambda i, h: taps.append(h.clone()))
        eng.close(s)
        eng.check()
        tally.add(got, o.logits(toks), (name, n))
        if n == 67:
            streams = []
            P.forward(o.cfg, o.w, toks, streams)
            assert len(taps) == 1 + len(streams) == 1 + len(o.cfg["layers"])
            assert rel(taps[0], P.norm(o.w["embed"].double()[toks], o.w["embed.norm"].double(), o.cfg["norm"]["eps"])) < 1e-6
            for i, (a, b) in enumerate(zip(taps[1:], streams)):
                t2 = Tally(dtype)
                t2.add(a, b, (name, "after layer", i))
                t2.close()
    tally.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first_token_equals_the_prompt_whole(folders, oracles, name, dtype):
    eng = engine(folders[name], dtype)
    toks = random_prompts(oracles[name].cfg["vocab"], [150], 7)[0]
    want = oracles[name].logits(toks)
    s, tally = eng.open(), Tally(dtype)
    for t, tok in enumerate(toks):
        tally.add(eng.step([(s, [tok])], want="last"), want[t:t + 1], t)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, cuts", [("A", [2, 62, 1, 3, 64, 18]), ("A", [39, 2, 2, 107]), ("A", [1, 1, 2, 146]), ("B", [128, 22]), ("B", [6, 2, 2, 2, 138]),
                                        ("C", [2, 2, 2, 3, 141]), ("C", [69, 2, 59, 2, 18]), ("D", [5, 60, 64, 2, 19]), ("D", [64, 64, 22]),
                                        ("B", [15, 2, 16, 2, 115]), ("C", [47, 48, 49, 6])])
def test_a_prompt_in_portions(folders, oracles, dtype, name, cuts):
    eng = engine(folders[name], dtype)
    toks = random_prompts(oracles[name].cfg["vocab"], [150], 9)[0]
    want = oracles[name].logits(toks)
    s, at, tally = eng.open(), 0, Tally(dtype)
    for c in cuts:
        tally.add(eng.step([(s, toks[at:at + c])], want="all"), want[at:at + c], (at, c))
        at += c
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_in_one_batch_then_decoded_together_and_slots_used_again(folders, oracles, name, dtype):
    o = oracles[name]
    eng, vocab = engine(folders[name], dtype, max_tokens=64 * 12, max_slots=4), o.cfg["vocab"]
    cut = [3, 70, 1, 129]
    prompts = random_prompts(vocab, [c + m for c, m in zip(cut, (4, 9, 2, 12))], 21)
    want = [o.logits(p) for p in prompts]
    slots = [eng.open() for _ in prompts]
    lg = eng.step([(s, p[:c]) for s, p, c in zip(slots, prompts, cut)], want="all")
    off, tally = 0, Tally(dtype)
    for i, (p, c, w) in enumerate(zip(prompts, cut, want)):
        tally.add(lg[off:off + c], w[:c], ("prompt", i))
        off += c
    live, t = list(range(4)), 0
    while live:
        lg = eng.step([(slots[i], [prompts[i][cut[i] + t]]) for i in live], want="last")
        for j, i in enumerate(live):
            tally.add(lg[j:j + 1], want[i][cut[i] + t:cut[i] + t + 1], (i, t))
        t += 1
        for i in list(live):
            if cut[i] + t == len(prompts[i]):
                eng.close(slots[i])                                  # the shorter requests end earlier
                live.remove(i)
    assert all(n == 0 for n in eng.cache.pages_in_use())
    # the freed slots (state areas) and pages serve other requests; what they held before must not show
    again = random_prompts(vocab, [66, 5, 1], 22)
    slots = [eng.open() for _ in again]
    lg = eng.step(list(zip(slots, again)), want="all")
    for a, b, p in ((0, 66, again[0]), (66, 71, again[1]), (71, 72, again[2])):
        tally.add(lg[a:b], o.logits(p), "slot used again")
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_long_decoding_across_page_borders_and_past_every_window(folders, oracles, name, dtype):
    eng = engine(folders[name], dtype)
    toks = random_prompts(oracles[name].cfg["vocab"], [5 + 215], 31)[0]
    want = oracles[name].logits(toks)
    s, tally = eng.open(), Tally(dtype)
    eng.step([(s, toks[:5])], want=None)
    for t in range(5, len(toks)):
        tally.add(eng.step([(s, [toks[t]])], want="last"), want[t:t + 1], t)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_just_inside_and_just_outside_the_reach_of_window_and_convolution(tmp_path, dtype):
    """One attention layer alone, a window of 45 behind a convolution of three taps: a position's logits depend on the token
    44 + 2 back (through the convolution of the oldest key) and not on the one 47 back, in a prompt and decoded, with the edge
    inside a page and on its border."""
    from megerax_tiny import _att, _layer
    cfg = {"architecture": "Megerax", "vocab": 90, "width": 64, "logit_scale": 1.0, "norm": {"eps": 1e-6},
           "layers": [_layer("attention", _att(4, 2, 32, 16, 3, 0.05, 30.0, 16, 10000.0, 45), None)]}
    folder = make_megerax_folder(tmp_path, "edge", cfg=cfg, seed=3)
    o, eng = Oracle(folder), engine(folder, dtype, max_tokens=64 * 8, max_slots=2)
    toks = random_prompts(90, [200], 4)[0]
    for j in (81, 100):                                                      # the places of a changed token
        other = list(toks)
        other[j] = (toks[j] + 7) % 90
        wa, wb = o.logits(toks), o.logits(other)
        assert (wa[j + 46] - wb[j + 46]).abs().max().item() > 1e-3 and torch.equal(wa[j + 47:], wb[j + 47:])
        for cut in (j + 40, j + 46, j + 47):                                 # decoded from just before the edge, at it, and past it
            rows = []
            for seq in (toks, other):
                s = eng.open()
                got = [eng.step([(s, seq[:cut])], want="all")]
                got += [eng.step([(s, [t])], want="last") for t in seq[cut:j + 52]]
                rows.append(torch.cat(got))
                eng.close(s)
            d = (rows[0] - rows[1]).abs().amax(-1).cpu()
            assert d[j + 46].item() > 1e-4 and d[j + 47:].max().item() == 0, (j, cut)
            tally = Tally(dtype)
            tally.add(rows[1], wb[:j + 52], (j, cut))
            tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "D"])
def test_a_token_far_back_still_counts(folders, oracles, name, dtype):
    """Two prompts that differ in their first token only: 300 tokens on the logits still differ (through the matrices of state, and
    in A through the latent, which every position sees), and the engine follows the plain implementation on both."""
    o = oracles[name]
    a = random_prompts(o.cfg["vocab"], [310], 77)[0]
    b = [(a[0] + 1) % o.cfg["vocab"]] + a[1:]
    wa, wb = o.logits(a), o.logits(b)
    assert rel(wa[290:], wb[290:]) > 5e-4
    eng, got = engine(folders[name], dtype), []
    for toks, want in ((a, wa), (b, wb)):
        s, tally = eng.open(), Tally(dtype)
        tally.add(eng.step([(s, toks[:200])], want="all"), want[:200])
        tally.add(eng.step([(s, toks[200:296])], want="all"), want[200:296])
        rows = [eng.step([(s, [toks[t]])], want="last") for t in range(296, 310)]
        tally.add(torch.cat(rows), want[296:310])
        got.append(torch.cat(rows))
        tally.close()
        eng.close(s)
    if dtype == "float32":                                                   # the difference itself, not only each side
        assert rel(got[0] - got[1], wa[296:310] - wb[296:310]) < 0.05
    eng.check()


@pytest.mark.parametrize("what", ["sink", "q.conv", "k.conv", "v.conv", "q.b", "k.b", "v.b", "q.norm", "k.norm", "dq.norm", "dkv.norm", "mix.norm", "mix.g",
                                  "mix.b", "A_log", "dt_bias", "a2", "g2", "embed.norm", "norm1"])
def test_every_small_tensor_counts_in_the_model(folders, oracles, what):
    """The plain implementation with one kind of tensor neutral gives other logits than the model's by far more than the tolerance;
    the engine, which meets the tolerance on the model's own, therefore reads it."""
    o = oracles["A"]
    toks = random_prompts(o.cfg["vocab"], [90], 5)[0]
    want, w = o.logits(toks), dict(o.w)
    for n, t in o.w.items():
        if n.endswith("." + what) or n == what:
            if what.endswith("conv"):
                w[n] = torch.zeros_like(t)
                w[n][:, -1] = 1.0
            elif what == "sink":
                w[n] = torch.full_like(t, -1e4)
            else:
                w[n] = torch.ones_like(t) if "norm" in what else torch.zeros_like(t)
    assert rel(P.forward(o.cfg, w, toks), want) > 0.01
    eng = engine(folders["A"], "float32")
    s, tally = eng.open(), Tally("float32")
    tally.add(eng.step([(s, toks)], want="all"), want)
    tally.close()
    eng.check()


@pytest.mark.parametrize("path, value", [("logit_scale", 0.5), ("norm.eps", 1e-2), ("layers.0.mixer.softcap", 3.0), ("layers.0.mixer.scale", 0.1),
                                         ("layers.0.mixer.mask.size", 41), ("layers.0.mixer.rot.base", 500.0), ("layers.0.mixer.rot.scaling.factor", 2.0),
                                         ("layers.0.mixer.rot.scaling.low", 0.1), ("layers.0.mixer.rot.scaling.high", 30.0),
                                         ("layers.0.mixer.rot.scaling.original", 512), ("layers.2.mixer.scale", 0.1), ("layers.2.mixer.rot.base", 20.0),
                                         ("layers.3.mixer.softcap", 2.0), ("layers.3.mixer.mask.size", 10), ("layers.3.mixer.mask.size", 90)])
def test_every_constant_of_the_configuration_counts(tmp_path, folders, oracles, path, value):
    cfg = json.loads(json.dumps(oracles["A"].cfg))
    both = [path] + [path.replace("layers.0", "layers.3")] if "rot" in path and "layers.0" in path else [path]     # a reader's rotation is its owner's
    for p in both:
        cur, keys = cfg, p.split(".")
        for k in keys[:-1]:
            cur = cur[int(k)] if k.isdigit() else cur[k]
        cur[keys[-1]] = value
    o = oracles["A"]
    toks = random_prompts(cfg["vocab"], [110], 5)[0]
    want = P.forward(cfg, o.w, toks)
    assert rel(want, o.logits(toks)) > 2e-3
    from braidinfer_b200.engine import Engine
    eng = Engine(cfg, {n: t for n, t in o.w.items()}, dtype="float32", max_tokens=64 * 4, verbose=False)
    s, tally = eng.open(), Tally("float32")
    tally.add(eng.step([(s, toks)], want="all"), want)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", list(range(1, 15)))
def test_configurations_drawn_from_a_seed(tmp_path, seed, dtype):
    """Other sizes, head counts, layer orders and constants than any written by hand: a prompt in two portions beside a second
    request, then both decoded together, against the plain implementation."""
    cfg = random_config(seed)
    folder = make_megerax_folder(tmp_path, f"r{seed}", cfg=cfg, seed=100 + seed)
    oracle, eng = Oracle(folder), engine(folder, dtype, max_tokens=64 * 8, max_slots=3)
    a, b = random_prompts(cfg["vocab"], [150, 21], seed)
    wa, wb = oracle.logits(a), oracle.logits(b)
    sa, sb, tally = eng.open(), eng.open(), Tally(dtype)
    tally.add(eng.step([(sa, a[:3])], want="all"), wa[:3], "first tokens")
    lg = eng.step([(sa, a[3:135]), (sb, b[:9])], want="all")
    tally.add(lg[:132], wa[3:135], "portion")
    tally.add(lg[132:], wb[:9], "beside it")
    for t in range(12):
        lg = eng.step([(sa, [a[135 + t]]), (sb, [b[9 + t]])], want="last")
        tally.add(lg[:1], wa[135 + t:136 + t], ("decoded", t))
        tally.add(lg[1:], wb[9 + t:10 + t], ("decoded beside", t))
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_the_library_entry_point(folders, oracles, name, dtype):
    import braidinfer_b200 as lib
    o = oracles[name]
    model = lib.load(folders[name], dtype=dtype, max_seq_len=256, max_batch=3, verbose=False)
    prompts = random_prompts(o.cfg["vocab"], [4, 61, 17, 9], 51)          # four requests, three slots
    outs = model.generate(prompts, lib.SamplingParams.greedy(), stop_tokens=(), max_new_tokens=[6, 8, 3, 5])
    for p, out, n in zip(prompts, outs, [6, 8, 3, 5]):
        assert len(out.tokens) == n
        toks = list(p)
        for t in out.tokens:
            row = o.logits(toks)[-1]
            if dtype == "float32":
                assert t == argmax_lowest(row)
            else:
                assert row[t] >= row.max() - 2 * TOL[dtype] * row.abs().max()
            toks.append(t)
    model.engine.check()


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_graphs_and_fused_sums_on_and_off(folders, oracles, name):
    """CUDA graphs change no bit; a product whose partial sums the next norm adds up gives what the plain reduce gives."""
    toks = random_prompts(oracles[name].cfg["vocab"], [40], 5)[0]
    res = {}
    for graphs, fused in ((True, True), (False, True), (True, False)):
        eng = engine(folders[name], "bfloat16", use_graphs=graphs, fuse_reduce=fused)
        s = eng.open()
        out = [eng.step([(s, toks[:20])], want="last")]
        out += [eng.step([(s, [t])], want="last") for t in toks[20:]]
        res[graphs, fused] = torch.cat(out)
        if graphs:
            assert eng.graph_replays > 10
        eng.check()
    assert torch.equal(res[True, True], res[False, True])
    assert rel(res[True, False], res[True, True].cpu()) < 1e-2


def test_logits_do_not_depend_on_the_batch_or_on_the_cut_beyond_rounding(folders, oracles):
    """float32: the same request alone and whole, beside others, and cut in portions gives logits equal to a few
    units in the last place of the sums."""
    eng = engine(folders["A"], "float32", max_slots=4)
    a, b, c = random_prompts(oracles["A"].cfg["vocab"], [90, 7, 130], 3)
    s = eng.open()
    alone = eng.step([(s, a)], want="all")
    eng.close(s)
    sa, sb, sc = eng.open(), eng.open(), eng.open()
    lg = eng.step([(sb, b), (sa, a[:50]), (sc, c)], want="all")
    part = [lg[7:57]]
    lg = eng.step([(sb, [1]), (sa, [a[50]]), (sc, [2])], want="last")
    part.append(lg[1:2])
    eng.close(sb)
    part.append(eng.step([(sa, a[51:]), ], want="all"))
    assert rel(torch.cat(part), alone.cpu()) < 2e-5
    eng.check()


def test_trace_replay_program_on_a_model_folder(folders, oracles, tmp_path):
    import numpy as np
    toks = random_prompts(oracles["A"].cfg["vocab"], [40, 9], 61)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[0][:33], "want": [0, 32]}, {"id": "b", "tokens": toks[1][:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [toks[0][33]], "want": [0]}, {"id": "b", "tokens": [toks[1][8]], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [toks[0][34]], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[0][35:], "want": [4]}], "end": ["a"]}]
    o = oracles["A"]
    vocab, wa, wb = o.cfg["vocab"], o.logits(toks[0]), o.logits(toks[1])
    for dtype in DTYPES:
        out = tmp_path / dtype
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders["A"], "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps).encode(),
                           capture_output=True, timeout=600)
        assert p.returncode == 0, p.stderr.decode()[-2000:]
        assert [l for l in p.stdout.decode().split("\n") if l.startswith("done")] == [f"done {i}" for i in range(4)]
        got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, vocab)) for i in (0, 1, 3)}
        assert not (out / "2.f32").exists()
        tol = TOL[dtype] * (1 if dtype == "float32" else 2)
        assert rel(got[0], wa[[0, 32]]) < tol and rel(got[1], torch.stack([wa[33], wb[8]])) < tol
        assert rel(got[3], wa[39:40]) < tol


def test_generate_command_line_on_a_model_folder(folders, oracles):
    env = dict(os.environ, MODEL=folders["B"], MAX_TOKENS="6", RAW="1", DTYPE="float32", MAX_SEQ_LEN="128")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "7, 200, 31, 4"], env=env, capture_output=True,
                       text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    toks, want = [7, 200, 31, 4], []
    for _ in range(6):
        t = argmax_lowest(oracles["B"].logits(toks)[-1])
        want.append(t)
        toks.append(t)
    assert [int(x) for x in p.stdout.split()] == want
