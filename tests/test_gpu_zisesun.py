"""Zisesun on the GPU: every new kernel alone against plain float64 formulas, then the whole model through the
engine (prompts whole, in portions, token by token, in unequal batches, with slots and pages used again, long
decoding, greedy generation, trace replay, the command line) against tests/plain_zisesun.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_zisesun as P
from test_gpu_birepel import argmax_lowest, paged
from test_gpu_loduzen import DTYPES, ROOT, TOL, TORCH, Tally, back, dev, engine, rel, step_tables
from tiny import random_prompts, read_weights
from zisesun_tiny import ZS_CONFIGS, folder_config, make_zisesun_folder, random_config

pytestmark = pytest.mark.gpu
D = torch.float64


@pytest.fixture(scope="module")
def K():
    from braidinfer_b200.csrc.api import get_kernels
    return get_kernels(verbose=False)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    base = tmp_path_factory.mktemp("zisesun")
    d = {n: make_zisesun_folder(base, n) for n in ZS_CONFIGS}
    d.update({n + "~": make_zisesun_folder(base, n, steady=True) for n in ZS_CONFIGS})
    return d


def fold(name, dtype):
    """The folder a run of this precision reads: a bfloat16 run takes the one whose experts rest on no close call (named with
    a tilde), since one expert chosen otherwise moves a position by far more than rounding does."""
    return name if dtype == "float32" else name + "~"


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


# ================================================================== kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("nqh, nkh, dk, dv, biased, normed, unit_v", [
    (4, 2, 32, 48, True, True, True), (3, 3, 40, 40, True, True, True), (2, 1, 64, 64, False, True, True), (8, 2, 8, 24, True, False, True),
    (6, 2, 24, 8, True, True, False), (3, 1, 20, 12, True, True, True), (1, 1, 5, 7, True, True, True), (2, 1, 256, 136, True, True, True),
    (16, 4, 128, 128, True, True, True), (5, 5, 16, 16, True, False, False)])
def test_biases_whole_projection_norms_unit_values_and_cache_write(K, dtype, nqh, nkh, dk, dv, biased, normed, unit_v):
    g = torch.Generator().manual_seed(dk + dv)
    page, eps = 64, 1e-5
    hd = -(-max(dk, dv) // 16) * 16
    lengths, before = [3, 70, 1], [0, 60, 129]                   # positions 0.., across a page border, and far on
    t = step_tables(lengths, before, pad=2)
    nq, nk, nv = nqh * dk, nkh * dk, nkh * dv
    # heads of unlike sizes: a norm a head instead of one over all of them would show
    grow = torch.cat([torch.linspace(0.3, 3.0, nqh).repeat_interleave(dk), torch.linspace(3.0, 0.3, nkh).repeat_interleave(dk),
                      torch.linspace(0.5, 2.0, nkh).repeat_interleave(dv)])
    src = torch.randn(t.rows, nq + nk + nv, generator=g) * grow
    src = dev(torch.cat([src, torch.full((t.rows, -(nq + nk + nv) % 8 + 8), 5.0)], 1), dtype)
    bias = [dev(torch.randn(n, generator=g), dtype) for n in (nq, nk, nv)] if biased else None
    q_w, k_w = (dev(1 + 0.3 * torch.randn(n, generator=g), dtype) for n in (nq, nk)) if normed else (None, None)
    total = [b + n for b, n in zip(before, lengths)]
    table, cache = paged(total, nkh, page, hd, dtype, g)
    cache.fill_(7.0)
    q = torch.full((t.rows, nqh * hd), 7.0, dtype=TORCH[dtype], device="cuda")
    K.proj_prep_kv(src, q, t.positions, t.token_seq, table.cuda(), cache, nqh, nkh, dk, dv, hd, eps, q_w=q_w, k_w=k_w, biases=bias,
                   v_unit=unit_v)
    K.check_device_errors()
    x = back(src)[:, :nq + nk + nv]
    if biased:
        x = x + torch.cat([back(b) for b in bias])
    qs, ks, vs = x[:, :nq], x[:, nq:nq + nk], x[:, nq + nk:].view(-1, nkh, dv)
    if normed:
        qs, ks = P.unit(qs, eps) * back(q_w), P.unit(ks, eps) * back(k_w)
    if unit_v:
        vs = P.unit(vs, eps)
    qs, ks = qs.reshape(-1, nqh, dk), ks.reshape(-1, nkh, dk)
    tol, live = 3e-6 if dtype == "float32" else 6e-3, t.n_tokens
    got_q = back(q).view(-1, nqh, hd)
    assert rel(got_q[:live, :, :dk], qs[:live]) < tol and got_q[:live, :, dk:].abs().sum().item() == 0
    assert got_q[live:].abs().sum().item() == 0                                 # rows of padding ask for nothing
    pos, seq = t.positions.cpu(), t.token_seq.cpu()
    for r in range(live):
        pg, off = int(table[seq[r], pos[r] // page]), int(pos[r] % page)
        row = back(cache[pg, :, :, off])                                        # [2, nkh, hd]
        assert rel(row[0, :, :dk], ks[r]) < tol and rel(row[1, :, :dv], vs[r]) < tol, r
        assert row[0, :, dk:].abs().sum().item() == 0 and row[1, :, dv:].abs().sum().item() == 0
    assert (back(cache) != 7.0).any(-1).sum().item() == 2 * nkh * live          # no other place of the cache was touched


def plain_biased_attention(q, keys, vals, pos, scale, r1, r2, nkh, size):
    """q [n, H, hd] at positions pos over keys, vals [total, G, hd]: behind a window, a distance bias a head."""
    n, H, _ = q.shape
    j = torch.arange(keys.shape[0])[None, :]
    vis = (j <= pos[:, None]) & (pos[:, None] - j < size)
    d = (pos[:, None] - j).clamp_min(0)
    out = torch.zeros(n, H, vals.shape[-1], dtype=D)
    for a in range(H):
        c = a // (H // nkh)
        s = (q[:, a] @ keys[:, c].T) * scale - P.distance_bias(d, torch.zeros_like(d), r1[a], r2[a])
        out[:, a] = P.softmax(s, vis) @ vals[:, c]
    return out


@pytest.mark.parametrize("kernel", ["simple_f32", "simple_bf16", "mma_prompt", "mma_few_1", "mma_few_7", "tcgen05_prompt"])
@pytest.mark.parametrize("nqh, nkh, hd, size", [(4, 2, 48, 40), (6, 3, 16, 64), (3, 3, 48, 7), (8, 1, 64, 70), (4, 4, 128, 96), (2, 1, 64, 300),
                                                (2, 2, 32, 1), (4, 1, 128, 65), (6, 2, 64, 127), (5, 1, 96, 1000)])
def test_attention_with_a_distance_bias_behind_a_window(K, kernel, nqh, nkh, hd, size):
    """For the last query of each sequence three keys stand out alike, with large values: the oldest one inside the window, the one
    just outside, and the query's own.  One key let in or left out by mistake, or a bias that does not tell the far one from
    the near one, moves that row by a large part of itself."""
    if kernel == "tcgen05_prompt" and hd not in (64, 128):
        pytest.skip("the tcgen05 kernel takes heads of 64 and 128")
    g = torch.Generator().manual_seed(nqh * hd + size)
    dtype = "float32" if kernel == "simple_f32" else "bfloat16"
    few = kernel.startswith("mma_few")
    n_few = int(kernel[-1]) if few else 0
    lengths, before = ([n_few, 1], [320 - n_few, 131]) if few else ([150, 37], [0, 290])
    t = step_tables(lengths, before, pad=1)
    total = [b + n for b, n in zip(before, lengths)]
    page, scale = 64, 0.35
    table, cache = paged(total, nkh, page, hd, dtype, g)
    keys, vals = [torch.randn(n, nkh, hd, generator=g) for n in total], [torch.randn(n, nkh, hd, generator=g) for n in total]
    u = torch.zeros(hd)
    u[hd // 2] = 1.0                                                         # every query leans this way; planted keys too
    for s in range(2):
        for j in {total[s] - 1 - size, total[s] - size, total[s] - 1}:
            if j >= 0:
                keys[s][j] = 12.0 * u
                vals[s][j] = 5.0 * torch.sign(torch.randn(nkh, hd, generator=g))
        for j in range(total[s]):
            pg = int(table[s, j // page])
            cache[pg, 0, :, j % page] = dev(keys[s][j], dtype)
            cache[pg, 1, :, j % page] = dev(vals[s][j], dtype)
    q0 = torch.randn(t.rows, nqh * hd + 8, generator=g)
    q0[:, :nqh * hd] += (4.0 * u).repeat(nqh)
    q = dev(q0, dtype)
    r1, r2 = torch.rand(nqh, generator=g) * 1.5 + 1.0, torch.rand(nqh, generator=g) * 0.6 + 0.05
    r1[0] = 0.02                                                             # a head that hardly minds the distance
    out = torch.full((t.rows, nqh * hd), 7.0, dtype=TORCH[dtype], device="cuda")
    kw = dict(distance_bias=(r1.cuda(), r2.cuda()))
    if kernel.startswith("simple"):
        K.attn_simple(q, out, cache, table.cuda(), t.positions, t.token_seq, nqh, nkh, hd, page, size, scale, **kw)
    elif kernel == "tcgen05_prompt":
        K.attn_tc(q, out, cache, table.cuda(), t.q_start, t.q_len, t.kv_before, 2, max(lengths), nqh, nkh, hd, size, scale, **kw)
    else:
        K.attn_mma(q, out, cache, table.cuda(), t.q_start, t.q_len, t.kv_before, t.token_seq, t.n_seqs, t.max_q_len, nqh, nkh, hd, size,
                   scale, n_splits=1 if not few else 3 if size > 128 else 2, few_tokens=few, **kw)
    K.check_device_errors()
    qs, r0, shown = back(q)[:, :nqh * hd].view(-1, nqh, hd), 0, [0.0, 0.0, 0.0]
    for s in range(2):
        rows = slice(r0, r0 + lengths[s])
        pos = torch.arange(before[s], total[s])
        kk, vv = back(dev(keys[s], dtype)), back(dev(vals[s], dtype))
        want = plain_biased_attention(qs[rows], kk, vv, pos, scale, r1.double(), r2.double(), nkh, size)
        assert rel(back(out)[rows].view(-1, nqh, hd), want) < (2e-5 if dtype == "float32" else 3e-2), (kernel, s)
        for i, (f1, f2, sz) in enumerate(((1.0, 1.0, size + 1), (1.0, 1.0, max(size - 1, 1)), (0.0, 1.0, size))):    # what faults would give
            other = plain_biased_attention(qs[rows], kk, vv, pos, scale, f1 * r1.double(), f2 * r2.double(), nkh, sz)
            shown[i] = max(shown[i], rel(other, want))
        r0 += lengths[s]
    if size < min(total):
        assert shown[0] > 0.15 and (size == 1 or shown[1] > 0.15)             # the test's inputs do show a window off by one
    assert size == 1 or shown[2] > 0.1                                        # and a bias that is left out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dk, dv, decays", [(24, 40, (0.4, 0.95, 0.998)), (136, 8, (0.8, 0.9995)), (8, 24, (0.996,)), (48, 70, (0.3, 0.9, 0.99, 1.0)),
                                            (256, 16, (0.97,)), (16, 16, (0.0, 0.5)), (128, 128, (0.9, 0.999))])
def test_lightning_whole_in_portions_and_token_by_token(K, dtype, dk, dv, decays):
    """Recurrence, norm over all heads and gate as the mixer chains them, with the states of two sequences kept in slots."""
    g = torch.Generator().manual_seed(dk + dv)
    H, eps, lens = len(decays), 1e-5, [41, 7]
    w, dec = dev(1 + 0.3 * torch.randn(H * dv, generator=g), dtype), torch.tensor(decays).cuda()
    seqs, want = [], []
    for n in lens:
        q, k = [dev(torch.randn(n, H * dk, generator=g), dtype) for _ in range(2)]
        v, gate = [dev(torch.randn(n, H * dv, generator=g), dtype) for _ in range(2)]
        seqs.append((q, k, v, gate))
        sq, sk, sv = (P.silu(back(x)) for x in (q, k, v))
        walks = [P.decayed_memory(sq[:, a * dk:(a + 1) * dk], sk[:, a * dk:(a + 1) * dk], sv[:, a * dv:(a + 1) * dv], float(dec[a])) for a in range(H)]
        o = torch.stack([x[0] for x in walks], 1)
        want.append((P.unit(o.reshape(n, H * dv), eps) * back(w) * P.sigmoid(back(gate)), torch.stack([x[1] for x in walks])))
    tol = 2e-5 if dtype == "float32" else 6e-3
    for cuts in ([[41, 7]], [[1, 1], [2, 2], [38, 4]], [[20, 0], [1, 7], [20, 0]], [[3, 2], [38, 5]], [[1, 1]] * 7 + [[34, 0]]):
        state = torch.full((4, H * dk * dv * 4), 255, dtype=torch.uint8, device="cuda")    # what an earlier sequence left
        at = [0, 0]
        for cut in cuts:
            live = [i for i in range(2) if cut[i]]
            t = step_tables([cut[i] for i in live], before=[at[i] for i in live], slots=[[3, 1][i] for i in live], pad=2)
            for i in live:
                if at[i] == 0:
                    state[[3, 1][i]].zero_()                                  # the manager hands a new sequence a cleared slot
            q, k, v, gate = (torch.cat([seqs[i][j][at[i]:at[i] + cut[i]] for i in live] + [seqs[0][j][:2] * 0]) for j in range(4))
            o = torch.empty(t.rows, H * dv, dtype=torch.float32, device="cuda")
            K.linear_scan(q, k, v, dec, None, o, state, 0, t, H, H, dk, dv, "constant", act_silu=True)
            out = torch.full((t.rows, H * dv), 3.0, dtype=TORCH[dtype], device="cuda")
            K.gated_norm(o, gate, w, out, t.token_seq, H * dv, False, eps, gate_sigmoid=True)
            assert (out[t.n_tokens:] == 3.0).all()                            # rows of padding are left alone
            r = 0
            for i in live:
                assert rel(out[r:r + cut[i]], want[i][0][at[i]:at[i] + cut[i]]) < tol, (cuts, cut, i)
                r += cut[i]
                at[i] += cut[i]
        for slot, i in ((3, 0), (1, 1)):
            assert rel(state[slot].contiguous().view(torch.float32).view(H, dk, dv), want[i][1]) < 1e-5
        assert (state[[0, 2]] == 255).all()                                   # the other slots were not touched
    K.check_device_errors()


@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_of_a_long_prompt_keeps_a_token_from_its_start(K, dtype):
    """A prompt of 1,100 tokens, walked whole (chunks side by side with a carry between them) and in portions that end on, just
    before and just after the chunks' edges.  Key and value of one early token stand out by far and the decay is slow: every later
    read-out is that token's value, and a walk that lost it, or the state at an edge, returns something else."""
    H, dk, dv, n = 2, 32, 24, 1100
    g = torch.Generator().manual_seed(11)
    dec = torch.tensor([0.9995, 0.999]).cuda()
    q = dev(torch.randn(n, H * dk, generator=g).abs() + 0.5, dtype)            # queries of one sign: no read-out cancels
    k, v = (dev(torch.randn(n, H * d, generator=g) * 0.2, dtype) for d in (dk, dv))
    k[2], v[2] = 40.0, dev(20.0 * torch.rand(H * dv, generator=g), dtype)

    def plain(vals):
        sq, sk, sv = P.silu(back(q)), P.silu(back(k)), P.silu(vals)
        return torch.cat([P.decayed_memory(sq[:, a * dk:(a + 1) * dk], sk[:, a * dk:(a + 1) * dk], sv[:, a * dv:(a + 1) * dv], float(dec[a]))[0]
                          for a in range(H)], 1)

    want, other = plain(back(v)), back(v).clone()
    other[2] = 0.0
    assert rel(plain(other)[n - 1:], want[n - 1:]) > 0.5
    for cuts in ([1100], [128, 1, 63, 908], [127, 2, 971], [129, 127, 844], [2, 1098], [1024, 76], [1023, 1, 76]):
        state = torch.zeros(1, H * dk * dv * 4, dtype=torch.uint8, device="cuda")
        at = 0
        for cut in cuts:
            t, sl = step_tables([cut], before=[at]), slice(at, at + cut)
            o = torch.empty(cut, H * dv, dtype=torch.float32, device="cuda")
            K.linear_scan(q[sl], k[sl], v[sl], dec, None, o, state, 0, t, H, H, dk, dv, "constant", act_silu=True)
            assert rel(o, want[sl]) < 2e-5, (cuts, cut)                        # float32 from the projections on, in every run
            at += cut
    K.check_device_errors()


@pytest.mark.parametrize("experts, top", [(5, 2), (1, 1), (4, 4), (16, 1), (40, 6), (300, 8)])
def test_routing_with_a_correction_keeps_the_softmax_scores_as_weights(K, experts, top):
    g = torch.Generator().manual_seed(experts)
    logits = (torch.randn(33, experts, generator=g) * 2).cuda()
    for corr in (0.4 * torch.randn(experts, generator=g), -5.0 - torch.rand(experts, generator=g), torch.zeros(experts)):
        for renorm in (False, True):
            idx = torch.empty((33, top), dtype=torch.int32, device="cuda")
            wgt = torch.empty((33, top), dtype=torch.float32, device="cuda")
            K.moe_route(logits, idx, wgt, 1, 1, renorm=renorm, correction=corr.cuda())
            wi, ww = P.route(back(logits), corr.double(), top)
            s = torch.softmax(back(logits), -1) + corr.double()
            got = torch.gather(s, 1, idx.cpu().long())
            assert torch.allclose(got, torch.gather(s, 1, wi), atol=1e-6)       # as good a choice, should two be nearly tied
            mine = torch.gather(torch.softmax(back(logits), -1), 1, idx.cpu().long())
            assert rel(wgt, mine / mine.sum(-1, keepdim=True) if renorm else mine) < 2e-6
            assert all(len(set(r)) == top for r in idx.tolist())
    # without a correction or with the sum divided out the weights are others: the modes are told apart
    if 1 < top < experts:
        assert (P.route(back(logits), torch.zeros(experts, dtype=D), top)[1].sum(-1) < 0.999).any()


@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8, 11, 16])
@pytest.mark.parametrize("width, rows", [(96, 5), (100, 3), (101, 4), (1024, 3), (2112, 9), (4096, 2), (64, 300)])
def test_streams_written_mixed_read_and_normed(K, n, width, rows):
    """The write of one sublayer and the read of the next in one kernel, with the result as finished rows, as the partial sums of
    a stream-k product and as a token's experts left it, for every number of CTAs a row; and the ends of a model: streams that
    are all one row, and gathered rows whose streams are not written back."""
    g = torch.Generator().manual_seed(n * width)
    eps = 1e-5
    x = torch.randn(rows, n, width, generator=g).cuda()
    y = torch.randn(rows, width, generator=g).cuda()
    mix, back_, read = ((torch.randn(*s, generator=g)).cuda() for s in ((n, n), (n,), (n,)))
    X = back(x).transpose(0, 1)
    sources = {"rows": (y, back(y))}
    if width % 8 == 0 and width >= 64:
        xin = dev(torch.randn(rows, 256, generator=g), "bfloat16")
        wt = dev(torch.randn(width, 256, generator=g), "bfloat16")
        sources["partial"] = ((xin, wt), back(xin) @ back(wt).T)
    experts, top, tile = 6, min(3, n + 1), 16
    for dt in DTYPES:
        idx = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(rows)]).to(torch.int32).cuda()
        plan = K.moe_plan(idx, torch.zeros(rows, dtype=torch.int32).cuda(), experts, tile)
        slots = dev(torch.randn(plan[4] * tile, width, generator=g), dt)
        wgt = torch.rand(rows, top, generator=g).cuda()
        at = plan[1].cpu().view(rows, top).long()
        sources["experts " + dt] = ((slots, plan, wgt, top), (back(slots)[at] * back(wgt)[:, :, None]).sum(1))
    w = dev(1 + 0.3 * torch.randn(width, generator=g), "bfloat16")
    for name, (src, want_y) in sources.items():
        for cluster in (None, 1, 2, 4, 8):
            for out_dt in DTYPES:
                given = K.gemm_tc_partial(*src) if name == "partial" else src
                xo = torch.empty_like(x) if cluster == 2 else x.clone()
                out = torch.empty(rows, width, dtype=TORCH[out_dt], device="cuda")
                K.streams(x if cluster == 2 else xo, xo, n, y=given, mix=mix, back=back_, read=read, w=w, eps=eps, out=out, cluster=cluster)
                new = P.write_streams(X, back(mix), back(back_), want_y)
                u = P.read_streams(new, back(read))
                assert rel(xo.transpose(0, 1), new) < 5e-6, (name, cluster)
                assert rel(out, P.unit(u, eps) * back(w)) < (1e-5 if out_dt == "float32" else 6e-3), (name, cluster)
    # all streams one row; no result yet: nothing is written back
    one = torch.randn(rows, 1, width, generator=g).cuda()
    E = back(one).transpose(0, 1).expand(n, -1, -1)
    out = torch.empty(rows, width, device="cuda")
    if abs(back(read).sum().item()) > 0.05:
        K.streams(one, None, n, read=read, w=w.float(), eps=eps, out=out)
        assert rel(out, P.unit(P.read_streams(E, back(read)), eps) * back(w)) < 1e-4 / abs(back(read).sum().item())
    xo = torch.empty_like(x)
    K.streams(one, xo, n, y=y, mix=mix, back=back_, read=read, out=out)                      # no norm: the sum itself
    new = P.write_streams(E, back(mix), back(back_), back(y))
    assert rel(xo.transpose(0, 1), new) < 5e-6 and rel(out, P.read_streams(new, back(read))) < 1e-5
    # the end: rows gathered, the sum of the streams, the streams as they were
    pick = torch.randint(0, rows, (7,), generator=g).to(torch.int32).cuda()
    out, keep = torch.empty(7, width, device="cuda"), x.clone()
    K.streams(x, None, n, y=y, mix=mix, back=back_, w=w.float(), eps=eps, out=out, row_index=pick)
    total = P.write_streams(X, back(mix), back(back_), back(y)).sum(0)
    assert rel(out, (P.unit(total, eps) * back(w))[pick.cpu().long()]) < 1e-5 and torch.equal(x, keep)
    K.check_device_errors()


def test_the_streams_kernel_refuses_what_does_not_fit(K):
    from braidinfer_b200.csrc.api import KernelError
    x, y = torch.zeros(2, 3, 64, device="cuda"), torch.zeros(2, 64, device="cuda")
    m, v = torch.zeros(3, 3, device="cuda"), torch.zeros(3, device="cuda")
    for kw in (dict(y=y, mix=m[:2], back=v), dict(y=y[:1], mix=m, back=v), dict(y=y, mix=None, back=v), dict(out=torch.zeros(2, 32, device="cuda")),
               dict(out=torch.zeros(2, 64, device="cuda"), read=v[:2])):
        with pytest.raises(KernelError):
            K.streams(x, x, 3, **kw)
    with pytest.raises(KernelError):
        K.streams(torch.zeros(2, 17, 64, device="cuda"), None, 17, out=y)


# ================================================================== the whole model through the engine
NAMES = ["A", "B", "C", "D"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_every_layer(folders, oracles, name, dtype):
    o = oracles[fold(name, dtype)]
    eng, tally = engine(folders[fold(name, dtype)], dtype), Tally(dtype)
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
            for i, (a, b) in enumerate(zip(taps[1:], streams)):
                t2 = Tally(dtype)
                t2.add(a, b, (name, "after layer", i))
                t2.close()
            s = eng.open()
            again = eng.step([(s, toks)], want="all")                        # without a tap the streams are written by fewer kernels
            eng.close(s)
            assert rel(again, got.cpu()) < 1e-6
    tally.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_token_by_token_from_the_first_token_equals_the_prompt_whole(folders, oracles, name, dtype):
    eng = engine(folders[fold(name, dtype)], dtype)
    toks = random_prompts(oracles[fold(name, dtype)].cfg["vocab"], [150], 7)[0]
    want = oracles[fold(name, dtype)].logits(toks)
    s, tally = eng.open(), Tally(dtype)
    for t, tok in enumerate(toks):
        tally.add(eng.step([(s, [tok])], want="last"), want[t:t + 1], t)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, cuts", [("A", [2, 62, 1, 3, 64, 18]), ("A", [39, 2, 2, 107]), ("A", [1, 1, 2, 146]), ("B", [128, 22]), ("B", [6, 2, 2, 2, 138]),
                                        ("C", [2, 2, 2, 3, 141]), ("C", [69, 2, 59, 2, 18]), ("D", [5, 60, 64, 2, 19]), ("D", [64, 64, 22]), ("B", [15, 2, 16, 2, 115])])
def test_a_prompt_in_portions(folders, oracles, dtype, name, cuts):
    eng = engine(folders[fold(name, dtype)], dtype)
    toks = random_prompts(oracles[fold(name, dtype)].cfg["vocab"], [150], 9)[0]
    want = oracles[fold(name, dtype)].logits(toks)
    s, at, tally = eng.open(), 0, Tally(dtype)
    for c in cuts:
        tally.add(eng.step([(s, toks[at:at + c])], want="all"), want[at:at + c], (at, c))
        at += c
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_requests_in_one_batch_then_decoded_together_and_slots_used_again(folders, oracles, name, dtype):
    o = oracles[fold(name, dtype)]
    eng, vocab = engine(folders[fold(name, dtype)], dtype, max_tokens=64 * 12, max_slots=4), o.cfg["vocab"]
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
    again = random_prompts(vocab, [66, 5], 22)
    slots = [eng.open(), eng.open()]
    lg = eng.step([(slots[0], again[0]), (slots[1], again[1])], want="all")
    tally.add(lg[:66], o.logits(again[0]), "slot used again")
    tally.add(lg[66:], o.logits(again[1]), "slot used again")
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_long_decoding_across_page_borders_and_past_every_window(folders, oracles, name, dtype):
    eng = engine(folders[fold(name, dtype)], dtype)
    toks = random_prompts(oracles[fold(name, dtype)].cfg["vocab"], [5 + 215], 31)[0]
    want = oracles[fold(name, dtype)].logits(toks)
    s, tally = eng.open(), Tally(dtype)
    eng.step([(s, toks[:5])], want=None)
    for t in range(5, len(toks)):
        tally.add(eng.step([(s, [toks[t]])], want="last"), want[t:t + 1], t)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_token_just_inside_and_just_outside_the_reach_of_the_windows(tmp_path, dtype):
    """One attention layer alone behind a window of 45: a position's logits depend on the token 44 back and not on the one 45
    back, in a prompt and decoded, with the edge inside a page and on its border.  The changed token is given a value that no
    other has (its row of the embedding is far larger before the norm of values makes the sizes alike), so it shows."""
    cfg = {"architecture": "Zisesun", "vocab": 90, "width": 64, "streams": 2, "max_positions": 256, "norm": {"eps": 1e-6},
           "layers": [{"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 32, "vdim": 16, "scale": 0.05, "mask": {"size": 45}}, "mlp": None}]}
    folder = make_zisesun_folder(tmp_path, "edge", cfg=cfg, seed=3)
    o, eng = Oracle(folder), engine(folder, dtype, max_tokens=64 * 8, max_slots=2)
    toks = random_prompts(90, [200], 4)[0]
    far = [toks[k] for k in (83, 100)]
    for j in (83, 100):                                                      # the places of a changed token
        other = list(toks)
        other[j] = (toks[j] + 7) % 90
        wa, wb = o.logits(toks), o.logits(other)
        assert (wa[j + 44] - wb[j + 44]).abs().max().item() > 1e-3 and torch.equal(wa[j + 45:], wb[j + 45:])
        for cut in (j + 40, j + 44, j + 45):                                 # decoded from just before the edge, at it, and past it
            rows = []
            for seq in (toks, other):
                s = eng.open()
                got = [eng.step([(s, seq[:cut])], want="all")]
                got += [eng.step([(s, [t])], want="last") for t in seq[cut:j + 50]]
                rows.append(torch.cat(got))
                eng.close(s)
            d = (rows[0] - rows[1]).abs().amax(-1).cpu()
            assert d[j + 44].item() > 1e-3 and d[j + 45:].max().item() == 0, (j, cut)
            tally = Tally(dtype)
            tally.add(rows[1], wb[:j + 50], (j, cut))
            tally.close()
    assert len(set(far)) == 2
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "D"])
def test_a_token_far_back_still_counts_through_the_states(folders, oracles, name, dtype):
    """Two prompts that differ in their first token only: 300 tokens on the logits still differ (through the memories: every window
    has long passed), and the engine follows the plain implementation on both, in a prompt's portion and decoded."""
    o = oracles[fold(name, dtype)]
    a = random_prompts(o.cfg["vocab"], [310], 77)[0]
    b = [(a[0] + 1) % o.cfg["vocab"]] + a[1:]
    wa, wb = o.logits(a), o.logits(b)
    assert rel(wa[290:], wb[290:]) > 2e-3
    eng, got = engine(folders[fold(name, dtype)], dtype), []
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
        assert rel(got[0] - got[1], wa[296:310] - wb[296:310]) < 0.02
    eng.check()


@pytest.mark.parametrize("what", ["r1", "correction", "k.b", "v.b", "hc1.mix", "hc2.mix", "hc1.in", "hc2.out", "norm1", "pos", "mix.norm", "k.norm"])
def test_every_small_tensor_counts_in_the_model(folders, oracles, what):
    """The plain implementation with one kind of tensor neutral gives other logits than the model's by far more than the tolerance;
    the engine, which meets the tolerance on the model's own, therefore reads it."""
    o = oracles["A"]
    toks = random_prompts(o.cfg["vocab"], [90], 5)[0]
    want, w = o.logits(toks), dict(o.w)
    for n, t in o.w.items():
        if n.endswith("." + what) or n == what:
            w[n] = torch.zeros_like(t) if what in ("r1", "correction", "k.b", "v.b", "pos") else t.T.contiguous() if what.endswith(".mix") \
                else torch.full_like(t, t.mean().item()) if what.startswith("hc") else torch.ones_like(t)
    assert rel(P.forward(o.cfg, w, toks), want) > 0.01
    eng = engine(folders["A"], "float32")
    s, tally = eng.open(), Tally("float32")
    tally.add(eng.step([(s, toks)], want="all"), want)
    tally.close()
    eng.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8, 9, 10, 11, 12])
def test_configurations_drawn_from_a_seed(tmp_path, seed, dtype):
    """Other sizes, head counts, layer orders, stream counts and constants than any written by hand: a prompt in two portions
    beside a second request, then both decoded together, against the plain implementation."""
    cfg = random_config(seed)
    folder = make_zisesun_folder(tmp_path, f"r{seed}", cfg=cfg, seed=100 + seed, steady=dtype == "bfloat16")
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
    o = oracles[fold(name, dtype)]
    model = lib.load(folders[fold(name, dtype)], dtype=dtype, max_seq_len=256, max_batch=3, verbose=False)
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


def test_a_sequence_longer_than_the_table_of_positions_is_refused(folders, oracles):
    cfg = oracles["B"].cfg
    eng = engine(folders["B"], "bfloat16", max_tokens=64 * 8)
    toks = random_prompts(cfg["vocab"], [cfg["max_positions"] + 1], 1)[0]
    s = eng.open()
    eng.step([(s, toks[:-1])], want="last")
    eng.check()                                                      # the table's last row is still a position
    with pytest.raises(Exception):
        eng.step([(s, toks[-1:])], want="last")
        eng.check()


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_graphs_and_fused_sums_on_and_off(folders, oracles, name):
    """CUDA graphs change no bit; a product whose partial sums the streams kernel adds up gives what the plain reduce gives."""
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
    assert rel(res[True, False], res[True, True].cpu()) < 1e-6


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
    vocab = oracles["A"].cfg["vocab"]
    for dtype in DTYPES:
        o, out = oracles[fold("A", dtype)], tmp_path / dtype
        wa, wb = o.logits(toks[0]), o.logits(toks[1])
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folders[fold("A", dtype)], "--dtype", dtype,
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
