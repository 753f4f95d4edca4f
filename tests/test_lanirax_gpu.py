"""The Lanirax design in the engine against the plain implementation of tests/plain_lanirax.py.

Every test makes its own small configuration and random weights (tests/lanirax_cases.py, tests/lanirax_standout.py), writes a model
folder with the engine's random-weights mode, reads it back with the plain reader, and compares logits: float32 to 2e-4 of the
largest logit, bfloat16 to 6e-2 (tiny widths average little out).  In float32 the rows of every cut must also EQUAL the rows of
the whole request bit for bit: the 32-bit kernels take a token's sums in an order that depends on its position only.
"""
import os

import numpy as np
import pytest
import torch

import plain_lanirax as plain
from lanirax_cases import CASES, SINGLE, Harness, attention, config, pair, rel_err, write_model
from lanirax_standout import MARKER, ORDINARY, distance_model, window_model

pytestmark = pytest.mark.gpu
TOL = {"float32": 2e-4, "bfloat16": 6e-2}


def plain_logits(folder, tokens):
    cfg, w = plain.read_model(folder)
    return plain.forward(cfg, w, list(tokens)).numpy()


def plain_rows(folder, tokens, dtype):
    """The plain logits and which rows to compare.  In bfloat16 a token whose router's call is close (a gap below 0.05 between
    logits of size 2) may go to another expert, and its row then differs as a whole; such rows are left out.  float32 keeps every row."""
    cfg, w = plain.read_model(folder)
    margins = []
    want = plain.forward(cfg, w, list(tokens), margins=margins).numpy()
    clear = np.ones(len(tokens), dtype=bool)
    if dtype != "float32":
        for per_token in margins:
            clear &= np.array(per_token) >= 0.05
    return want, clear


def close(got, want, clear, dtype):
    """float32: every row.  bfloat16: the median row and nine of ten clear rows (a token that went to another expert also moves the
    keys and states that the rows after it read)."""
    rows = np.abs(got - want).max(axis=1) / np.abs(want).max()
    if dtype == "float32":
        return bool(rows.max() < TOL[dtype])
    rows = rows[clear]
    return bool((rows < TOL[dtype]).mean() >= 0.9 and np.median(rows) < 3e-2 and np.isfinite(got).all())


def tokens_of(rng, n, vocab):
    return rng.integers(0, vocab, n).tolist()


# ---- each mechanism alone: kernels -------------------------------------------------------------------------
@pytest.mark.parametrize("T, W", [(5, 48), (1, 36), (70, 257), (9, 512), (3, 260), (2, 4096)])
def test_the_norm_after_the_weighted_sum(T, W):
    """One output (with and without a bias it owes), one or two outputs normed first, the sum without a norm, and a token's experts'
    rows summed in the same kernel."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(T * 1000 + W)
    x, y0, y1 = torch.randn(T, W, generator=g), torch.randn(T, W, generator=g) * 3, torch.randn(T, W, generator=g) * 0.2
    w, w0, w1, bias = (1 + 0.2 * torch.randn(W, generator=g) for _ in range(4))
    d = lambda t: t.double()

    def run(outputs, **kw):
        xd, rounded = x.cuda(), torch.empty(T, W, dtype=torch.bfloat16, device="cuda")
        kw = {k: [t.cuda() for t in v] if isinstance(v, list) else v.cuda() if torch.is_tensor(v) else v for k, v in kw.items()}
        ops.residual_norm(xd, kw.pop("alpha", 1.7), [y.cuda() for y in outputs], kw.pop("weight", w.cuda()), 1e-3, rounded=rounded, **kw)
        assert torch.equal(rounded, xd.to(torch.bfloat16))
        return xd.cpu().double()

    same = lambda got, want: float((got - want).abs().max() / want.abs().max()) < 3e-6
    assert same(run([y0]), plain.rms_norm(1.7 * d(x) + d(y0), d(w), 1e-3))
    assert same(run([y0], bias=bias), plain.rms_norm(1.7 * d(x) + d(y0) + d(bias), d(w), 1e-3))
    n0, n1 = plain.rms_norm(d(y0), d(w0), 0.5), plain.rms_norm(d(y1), d(w1), 0.5)
    assert same(run([y0], member_weights=[w0], member_eps=0.5, factor=0.3), plain.rms_norm(1.7 * d(x) + 0.3 * n0, d(w), 1e-3))
    both = dict(member_weights=[w0, w1], member_eps=0.5, factor=0.5)
    assert same(run([y0, y1], **both), plain.rms_norm(1.7 * d(x) + 0.5 * (n0 + n1), d(w), 1e-3))
    assert same(run([y0, y1], weight=None, alpha=1.0, **both), d(x) + 0.5 * (n0 + n1))
    x.fill_(float("nan"))                                    # alpha 0: what x held is not read
    assert same(run([y0, y1], weight=None, alpha=0.0, **both), 0.5 * (n0 + n1))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W, top", [(5, 48, 3), (3, 257, 1), (6, 512, 7), (2, 2048, 4)])
def test_a_tokens_experts_summed_in_the_norms_kernel(T, W, top, dtype):
    """The same bits as the weighted sum and the norm in two kernels, and right."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(W + top)
    x, rows = torch.randn(T, W, generator=g), torch.randn(T * top + 5, W, generator=g).to(dtype)
    pair_row = torch.randperm(T * top + 5, generator=g)[:T * top].int()
    weights, w = torch.rand(T, top, generator=g), 1 + 0.1 * torch.randn(W, generator=g)
    one, two, y = x.cuda(), x.cuda(), torch.empty(T, W, device="cuda")
    ops.residual_norm_picks(one, 0.7, rows.cuda(), pair_row.cuda(), weights.cuda(), w.cuda(), 1e-5)
    ops.moe_combine(rows.cuda(), pair_row.cuda(), weights.cuda(), y)
    ops.residual_norm(two, 0.7, [y], w.cuda(), 1e-5)
    assert torch.equal(one, two)
    total = (rows.double()[pair_row.long()].reshape(T, top, W) * weights.double()[:, :, None]).sum(1)
    assert rel_err(one.cpu().numpy(), plain.rms_norm(0.7 * x.double() + total, w.double(), 1e-5).numpy()) < 3e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [36, 512, 1030, 4096])
def test_normed_embedding(W, dtype):
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(W)
    table, w = (torch.randn(11, W, generator=g) * 0.02).to(dtype), 1 + 0.2 * torch.randn(W, generator=g)
    toks = torch.tensor([3, 10, 0, 3, 7], dtype=torch.int32)
    x, rounded = torch.empty(5, W, device="cuda"), torch.empty(5, W, dtype=torch.bfloat16, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.embed_norm(table.cuda(), toks.cuda(), w.cuda(), x, status, 1e-3, 1.5, rounded)
    want = plain.rms_norm(table.double()[toks.long()] * 1.5, w.double(), 1e-3)
    assert int(status.item()) == 0 and rel_err(x.cpu().numpy(), want.numpy()) < 2e-6 and torch.equal(rounded, x.to(torch.bfloat16))
    ops.embed_norm(table.cuda(), torch.tensor([11], dtype=torch.int32, device="cuda"), w.cuda(), x[:1], status, 1e-3)
    assert int(status.item()) == 1                           # an id outside the vocabulary is flagged and reads nothing


def _paged(n, page, table_pages):
    """Device arrays of one sequence of ``n`` tokens in slot 1 whose pages lie in the given order."""
    table = torch.full((2, len(table_pages) + 1), -1, dtype=torch.int32)
    table[1, :len(table_pages)] = torch.tensor(table_pages, dtype=torch.int32)
    return table.cuda(), torch.tensor([1], dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")


@pytest.mark.parametrize("norm, weighted", [("before", True), ("after", False), ("after", True), ("none", False)])
@pytest.mark.parametrize("H, G, d, rd, pairing", [(4, 2, 16, 6, "interleaved"), (3, 1, 20, 20, "half"), (9, 3, 136, 70, "interleaved"),
                                                  (2, 2, 300, 34, "half"), (2, 1, 64, 0, "half"), (4, 2, 64, 28, "half"), (3, 1, 64, 30, "half"),
                                                  (2, 2, 64, 22, "interleaved"), (5, 1, 128, 128, "half"), (2, 2, 128, 72, "interleaved"),
                                                  (3, 3, 256, 96, "half"), (2, 1, 256, 90, "interleaved")])
def test_attention_operands(H, G, d, rd, pairing, norm, weighted):
    """Norm before and behind the rotation in both pairings, a factor per head and one per position, tied values."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(H + d + rd)
    n, page = 13, 4
    proj = torch.randn(n, (H + G) * d, generator=g)
    wq, wk = 1 + 0.2 * torch.randn(d, generator=g), 1 + 0.2 * torch.randn(d, generator=g)
    head, place = 1 + 0.3 * torch.rand(H, generator=g), 1 + 0.5 * torch.rand(40, generator=g)
    freqs, amp = plain.stretched_frequencies(rd, 90.0, {"factor": 3.0, "original": 300, "fast": 9.0, "slow": 2.0}) if rd else ([], 1.0)
    ang = torch.arange(40, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    cos, sin = ((ang.cos() * amp).float().cuda(), (ang.sin() * amp).float().cuda()) if rd else (None, None)
    table, slot, status = _paged(n, page, [3, 0, 5, 1])
    k_pool, v_pool = torch.full((6, G, page, d), float("nan"), device="cuda"), torch.full((6, G, page, d), float("nan"), device="cuda")
    q = torch.empty(n, H * d, device="cuda")
    pos, seq = torch.arange(n, dtype=torch.int32, device="cuda"), torch.zeros(n, dtype=torch.int32, device="cuda")
    ops.norm_rope_kvwrite(proj.cuda(), q, k_pool, v_pool, wq.cuda() if weighted else None, wk.cuda() if weighted else None, head.cuda(), cos, sin,
                          pos, seq, slot, table, status, 0, H * d, H * d, H, G, d, d, rd, page, 1e-2, norm=norm, pairing=pairing,
                          pos_scale=place.cuda())
    assert int(status.item()) == 0

    def rotate(x):
        if not rd:
            return x
        if pairing == "interleaved":
            order = list(range(d))
        else:                                                # element i with i + rd/2: the same rotation in another order
            order = [i // 2 + (i % 2) * (rd // 2) for i in range(rd)] + list(range(rd, d))
        y = plain.rotate_neighbours(x[..., order], {"dims": rd, "base": 90.0, "scaling": {"factor": 3.0, "original": 300, "fast": 9.0, "slow": 2.0}})
        out = torch.empty_like(y)
        out[..., order] = y
        return out

    def operand(x, w):
        if norm == "before":
            return rotate(plain.rms_norm(x, w.double(), 1e-2))
        y = rotate(x)
        if norm == "after":
            y = plain.unit_rms(y, 1e-2) * (w.double() if weighted else 1.0)
        return y
    x = proj.double()
    want_q = operand(x[:, :H * d].reshape(n, H, d), wq) * head.double()[None, :, None] * place.double()[:n, None, None]
    want_k = operand(x[:, H * d:].reshape(n, G, d), wk)
    assert rel_err(q.cpu().numpy(), want_q.reshape(n, -1).numpy()) < 3e-6
    at = lambda pool, p: pool[[3, 0, 5, 1][p // page], :, p % page].cpu().numpy()
    for p in range(n):
        assert rel_err(at(k_pool, p), want_k[p].numpy()) < 3e-6
        assert np.array_equal(at(v_pool, p), proj[p, H * d:].reshape(G, d).numpy())
    # a position past the table is flagged
    ops.norm_rope_kvwrite(proj[:1].cuda(), q[:1], k_pool, v_pool, None, None, None, None, None, pos[12:13], seq[:1], slot, table, status, 0, H * d,
                          H * d, H, G, d, d, 0, page, 1e-2, pos_scale=place[:12].contiguous().cuda())
    assert int(status.item()) == 3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H, G, d, dv, window, cap", [(4, 2, 16, 16, 0, 0.0), (8, 1, 32, 48, 11, 0.0), (3, 3, 12, 20, 0, 3.0), (4, 1, 64, 16, 40, 2.0)])
def test_attention_kernels_with_a_penalty_on_distance(H, G, d, dv, window, cap, dtype):
    """The float32-arithmetic kernel and, in bfloat16 with sizes it takes, the tensor-core kernel (single tokens and portions), with
    a cap on the scores, a window and a sink beside the penalty, on one sequence of 150 tokens of which the last come one by one."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(H * 7 + d)
    n, page = 150, 8
    pages = torch.randperm(20, generator=g)[:19].tolist()
    q, k, v = (torch.randn(n, h, s, generator=g).to(dtype) for h, s in ((H, d), (G, d), (G, dv)))
    slopes, sinks = torch.tensor([0.3 / 2 ** h for h in range(H)]), torch.randn(H, generator=g)
    table, slot, status = _paged(n, page, pages)
    k_pool = torch.zeros(20, G, page, d, dtype=dtype, device="cuda")
    v_pool = torch.zeros(20, G, page, dv, dtype=dtype, device="cuda")
    for p in range(n):
        k_pool[pages[p // page], :, p % page] = k[p].cuda()
        v_pool[pages[p // page], :, p % page] = v[p].cuda()
    scale = 1.5 / d ** 0.5
    dist = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).double()
    want = torch.zeros(n, H, dv, dtype=torch.float64)
    for h in range(H):
        s = (q[:, h].double() @ k[:, h // (H // G)].double().T) * scale
        s = cap * torch.tanh(s / cap) if cap else s
        s = (s - float(slopes[h]) * dist).masked_fill((dist < 0) | ((dist >= window) if window else (dist < 0)), float("-inf"))
        e = torch.exp(s)
        want[:, h] = (e @ v[:, h // (H // G)].double()) / (e.sum(-1, keepdim=True) + torch.exp(sinks[h].double()))
    want = want.reshape(n, -1).numpy()
    mma = dtype == torch.bfloat16 and ops.masked_attention_mma_supported(d, dv, H * d, d, d, dv, False)
    assert mma == (dtype == torch.bfloat16 and d % 16 == 0 and dv % 16 == 0)
    for kernel in ("plain", "mma") if mma else ("plain",):
        got = []
        for lo, hi in ((0, 97), (97, 99), *((p, p + 1) for p in range(99, n))):
            T = hi - lo
            pos = torch.arange(lo, hi, dtype=torch.int32, device="cuda")
            qd, out = q[lo:hi].reshape(T, -1).contiguous().cuda(), torch.empty(T, H * dv, dtype=dtype, device="cuda")
            if kernel == "plain":
                ops.masked_attention(qd, d, k_pool, v_pool, d, dv, None, out, pos, torch.zeros(T, dtype=torch.int32, device="cuda"), slot, table,
                                     status, H, G, d, dv, page, window, 0, scale, cap, sinks=sinks.cuda(), slopes=slopes.cuda())
            else:
                starts = torch.tensor([0, T], dtype=torch.int32, device="cuda")
                tiles = torch.tensor([[0, t] for t in range(0, T, 64)], dtype=torch.int32, device="cuda")
                ops.masked_attention_mma(qd, d, k_pool, v_pool, d, dv, None, out, pos, slot, starts, table, tiles, len(tiles), status, H, G, d, dv,
                                         page, window, 0, scale, cap, sinks=sinks.cuda(), slopes=slopes.cuda())
            got.append(out.float().cpu().numpy())
        assert int(status.item()) == 0
        assert rel_err(np.concatenate(got), want) < (1e-5 if dtype == torch.float32 else 2e-2), kernel


@pytest.mark.parametrize("E, top, K, gate", [(5, 2, 64, False), (8, 8, 96, True), (16, 4, 352, False), (33, 3, 512, True), (64, 6, 128, False),
                                             (100, 33, 64, False), (127, 5, 2048, True), (32, 4, 4096, False), (7, 2, 2080, True)])
def test_router_with_its_product_in_one_kernel(E, top, K, gate):
    """Against the plain router for every scoring, over full and part-filled blocks of tokens (with K of 2,048 and more and few tokens:
    several blocks that share K); a token's picks do not depend on the others."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(E + K)
    T, rows = 37, E + (1 if gate else 0)
    h = torch.randn(T, K, generator=g).to(torch.bfloat16)
    w = (torch.randn((rows + 3) // 4 * 4, K, generator=g) * 2 * K ** -0.5).to(torch.bfloat16)
    bias, corr = torch.randn(rows, generator=g) * 0.5, torch.randn(E, generator=g) * 0.1
    z = h.double() @ w.double()[:rows].T
    assert ops.moe_router_supported(h.cuda(), w.cuda(), rows)

    def run(sel=slice(None), **kw):
        n = h[sel].shape[0]
        ids, wts = torch.empty(n, top, dtype=torch.int32, device="cuda"), torch.empty(n, top, device="cuda")
        sg = torch.empty(n, device="cuda") if gate else None
        ops.moe_router(h[sel].contiguous().cuda(), w.cuda(), E, top, 1, 1, 1.0, ids, wts, sg, **kw)
        return ids.cpu(), wts.cpu(), sg.cpu() if gate else None

    for kw in ({"scoring": "softmax_chosen", "bias": bias.cuda()}, {"scoring": "softmax"}, {"scoring": "sigmoid", "correction": corr.cuda(), "renormalize": False}):
        ids, wts, sg = run(**kw)
        logits = z[:, :E] + (bias.double()[:E] if "bias" in kw else 0.0)
        score = torch.sigmoid(logits) if kw["scoring"] == "sigmoid" else torch.softmax(logits, dim=-1)
        choice = score + (corr.double() if "correction" in kw else 0.0)
        for t in range(T):
            order = torch.sort(choice[t], descending=True, stable=True).indices
            got = ids[t].long()
            assert len(set(got.tolist())) == top
            # (a call closer than the product's rounding may go either way)
            assert float(choice[t][order[:top]].min() - choice[t][got].min()) < 1e-5
            want = score[t][got] / (score[t][got].sum() if kw.get("renormalize", True) else 1.0)
            assert torch.allclose(wts[t].double(), want, rtol=2e-5, atol=1e-7)
        if gate:
            assert torch.allclose(sg.double(), torch.sigmoid(z[:, E]), atol=2e-6)
        for sel in (slice(0, 1), slice(17, 20), slice(36, 37)):
            a = run(sel, **kw)
            assert torch.equal(a[0], ids[sel]) and torch.equal(a[1], wts[sel])


@pytest.mark.parametrize("channel_decay", [False, True])
@pytest.mark.parametrize("H, G, d, dv, K", [(4, 2, 32, 24, 4), (2, 1, 64, 40, 5), (3, 3, 128, 16, 2), (2, 1, 256, 12, 3), (6, 2, 32, 7, 1)])
def test_delta_rule_kernels_with_key_heads_of_whole_warps(H, G, d, dv, K, channel_decay):
    """The convolution kernel that also makes unit keys: two sequences of 39 and 1 tokens in one step, then single tokens, then
    another portion; a token has the same bits however it was cut, and the values are right (decays per head and per channel)."""
    from carbon_engine_b200 import ops
    g = torch.Generator().manual_seed(H * 100 + d)
    n, C = 60, 2 * G * d + H * dv
    n_dec = H * d if channel_decay else H
    ld = (C + H + n_dec + H * dv + 3) // 4 * 4
    taps = torch.randn(C, K, generator=g) * 0.5
    a_log, dt_bias = torch.randn(H, generator=g) * 0.5, torch.randn(n_dec, generator=g) * 0.3
    norm_w = 1 + 0.1 * torch.randn(dv, generator=g)
    rows = [torch.randn(n, ld, generator=g) for _ in range(2)]
    mode = ops.DECAY_PER_CHANNEL if channel_decay else ops.DECAY_PER_HEAD

    def run(cuts):
        """cuts: per step, the tokens each sequence brings (0: left out)."""
        state = torch.zeros(3, H, d, dv, device="cuda")
        kept = torch.zeros(3, max(K - 1, 1), C, device="cuda")
        at, got = [0, 0], [[], []]
        for cut in cuts:
            who = [b for b in (0, 1) if cut[b]]
            lengths = [cut[b] for b in who]
            T = sum(lengths)
            seq = torch.tensor([i for i, m in enumerate(lengths) for _ in range(m)], dtype=torch.int32, device="cuda")
            starts = torch.tensor(np.concatenate([[0], np.cumsum(lengths)]), dtype=torch.int32, device="cuda")
            slots = torch.tensor([(2, 0)[b] for b in who], dtype=torch.int32, device="cuda")
            proj = torch.cat([rows[b][at[b]:at[b] + cut[b]] for b in who]).cuda()
            prep = torch.empty(T, ops.gated_delta_prep_width(H, G, d, dv, mode), device="cuda")
            raw, out = torch.empty(T, H * dv, device="cuda"), torch.empty(T, H * dv, device="cuda")
            ops.gated_delta(proj, proj[:, C + H:C + H + n_dec], proj[:, C + H + n_dec:C + H + n_dec + H * dv], taps.cuda(), a_log.cuda(),
                            dt_bias.cuda(), norm_w.cuda(), prep, raw, state, kept if K > 1 else None, out, seq, slots, starts, len(who), 0, C,
                            H, G, d, dv, K, 1e-5, decay=mode, gate=ops.GATE_SILU)
            i = 0
            for b in who:
                got[b].append(out[i:i + cut[b]].cpu())
                at[b] += cut[b]
                i += cut[b]
        return [torch.cat(x) for x in got]
    ops.reset_kernel_counts()
    a = run([(39, 1), (1, 1), (1, 0), (19, 58)])
    assert ops.kernel_counts()["gated_delta_conv_kernel"] == 4 and "gated_delta_prepare_kernel" not in ops.kernel_counts()
    b = run([(60, 0), (0, 60)])
    c = run([(2, 7), (5, 31), *[(1, 1)] * 22, (31, 0)])
    for i in range(2):
        assert torch.equal(a[i], b[i]) and torch.equal(a[i], c[i])
        x = rows[i].double()
        conv = plain.silu(plain.short_convolution(x[:, :C], taps.double()))
        q = plain.unit_length(conv[:, :G * d].reshape(n, G, d)) * d ** -0.5
        k = plain.unit_length(conv[:, G * d:2 * G * d].reshape(n, G, d))
        v, beta = conv[:, 2 * G * d:].reshape(n, H, dv), torch.sigmoid(x[:, C:C + H])
        dec = plain.softplus(x[:, C + H:C + H + n_dec] + dt_bias.double()).reshape(n, H, -1)
        dec = torch.exp(-torch.exp(a_log.double())[None, :, None] * dec).expand(n, H, d)
        want = torch.zeros(n, H, dv, dtype=torch.float64)
        for h in range(H):
            S = torch.zeros(d, dv, dtype=torch.float64)
            for t in range(n):
                S = dec[t, h][:, None] * S
                kk = k[t, h // (H // G)]
                S = S + torch.outer(kk, beta[t, h] * (v[t, h] - kk @ S))
                want[t, h] = q[t, h // (H // G)] @ S
        gate = plain.silu(x[:, C + H + n_dec:C + H + n_dec + H * dv])
        want = plain.rms_norm(want, norm_w.double(), 1e-5).reshape(n, -1) * gate
        assert rel_err(a[i].numpy(), want.numpy()) < 2e-5


def test_routing_with_a_bias_far_from_zero_and_equal_logits():
    """The bias joins the logits before the choice AND the softmax; equal logits go to the lower index; far logits do not overflow."""
    from carbon_engine_b200 import ops
    z = torch.tensor([[1.0, 2.0, 3.0, 0.0], [200.0, -300.0, 199.0, 5.0], [0.0, 0.0, 0.0, 0.0]])
    bias = torch.tensor([2.5, 0.0, -1.5, 0.0])
    ids, w = torch.empty(3, 2, dtype=torch.int32, device="cuda"), torch.empty(3, 2, device="cuda")
    ops.moe_route(z.cuda(), 4, 2, 1, 1, 1.0, ids, w, scoring="softmax_chosen", bias=bias.cuda())
    e = np.exp(1.5)
    assert ids.cpu().tolist() == [[0, 1], [0, 2], [0, 1]]
    assert np.allclose(w.cpu().numpy(), [[e / (e + 1), 1 / (e + 1)], [1 / (1 + np.exp(-5.0)), 1 / (1 + np.exp(5.0))],
                                         [1 / (1 + np.exp(-2.5)), 1 / (1 + np.exp(2.5))]], rtol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_silu_experts_products_over_the_layout_by_expert(dtype):
    """silu(gate) up in every product kernel: the FMA kernel, wmma and, in bfloat16, the grouped tcgen05 kernel in all its tiles."""
    from carbon_engine_b200 import ops, ops_tensor
    g = torch.Generator().manual_seed(3)
    ran = set()
    for T, E, top, K, ff, tile in ((9, 5, 2, 40, 24, 16), (70, 4, 3, 48, 31, 64), (33, 6, 2, 64, 80, 16), (200, 3, 2, 128, 136, 128), (90, 8, 4, 96, 64, 64)):
        h = torch.randn(T, K, generator=g).to(dtype)
        gate, up = (torch.randn(E, ff, K, generator=g).mul(2 * K ** -0.5).to(dtype) for _ in range(2))
        w = torch.stack([gate, up], dim=2).reshape(E, 2 * ff, K).contiguous()
        ids = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).int()
        tiles = ops.moe_max_tiles(T * top, E, tile)
        i32 = lambda n: torch.empty(n, dtype=torch.int32, device="cuda")
        row_token, pair_row, tile_expert, n_tiles = i32(tiles * tile), i32(T * top), i32(tiles), i32(1)
        ops.moe_align(ids.cuda(), E, tile, row_token, pair_row, tile_expert, n_tiles)
        z = torch.einsum("tk,efk->tef", h.double(), gate.double()), torch.einsum("tk,efk->tef", h.double(), up.double())
        want = plain.silu(z[0]) * z[1]
        outs = []
        if tile != 128:
            out = torch.zeros(tiles * tile, ff, dtype=dtype, device="cuda")
            ops.moe_matmul(h.cuda(), w.cuda(), out, tile, "silu_glu", row_token, tile_expert, n_tiles)
            outs.append(out)
        if ops_tensor.grouped_bf16_supported(tile, 2 * ff, K, K, ff, dtype):
            laid, out = torch.empty(tiles * tile, K, dtype=dtype, device="cuda"), torch.zeros(tiles * tile, ff, dtype=dtype, device="cuda")
            ops.moe_gather(h.cuda(), row_token, n_tiles, tile, laid)
            assert ops_tensor.grouped_bf16(laid, w.cuda(), out, tile, ops.MOE_ACTIVATIONS["silu_glu"], tile_expert, n_tiles)
            ran.add(tile)
            outs.append(out)
        for out in outs:
            got = out.float().cpu()[pair_row.cpu().long()].reshape(T, top, ff)
            ref = torch.stack([want[t, ids[t].long()] for t in range(T)])
            assert rel_err(got.numpy(), ref.numpy()) < (2e-6 if dtype == torch.float32 else 1e-2), (tile, T)
    assert ran == ({16, 64, 128} if dtype == torch.bfloat16 else set())


# ---- each mechanism alone: one layer -----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_one_layer_of_each_kind(tmp_path, name, dtype):
    folder = write_model(SINGLE[name], str(tmp_path / name), seed=7)
    toks = tokens_of(np.random.default_rng(5), 45, SINGLE[name]["vocab"])
    want, clear = plain_rows(folder, toks, dtype)
    h = Harness(folder, dtype)
    whole = h.run(toks)
    assert close(whole, want, clear, dtype)
    one_by_one = h.run(toks, [1])
    assert close(one_by_one, want, clear, dtype)
    if dtype == "float32":
        assert np.array_equal(whole, one_by_one)


def test_layers_outputs_one_after_another(tmp_path):
    """The residual after every layer run (a layer that runs another's weights counts), so that a fault shows where it is."""
    from carbon_engine_b200.engine.batch import StepEntry
    for name in ("A", "B"):
        folder = write_model(CASES[name], str(tmp_path / name))
        cfg, w = plain.read_model(folder)
        toks = tokens_of(np.random.default_rng(1), 30, cfg["vocab"])
        trace = []
        plain.forward(cfg, w, toks, trace)
        h = Harness(folder, "float32")
        rid = h.open()
        ctx, rows, commits = h.runner.prepare([StepEntry(rid, toks, [0])])
        got = []
        h.model.forward(ctx, h.storage, tap=lambda i, x: got.append(x.cpu().numpy().copy()))
        assert len(got) == len(trace) == 4
        for i, (a, b) in enumerate(zip(got, trace)):
            assert rel_err(a, b.numpy()) < 1e-4, (name, i)


# ---- whole models: cuts, batches, reuse ------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_whole_prompt_portions_and_decoding(tmp_path, name, dtype):
    from carbon_engine_b200 import ops
    folder = write_model(CASES[name], str(tmp_path / name), seed=11)
    big = name in ("T", "V")
    toks = tokens_of(np.random.default_rng(3), 150 if big else 83, CASES[name]["vocab"])
    want, clear = plain_rows(folder, toks, dtype)
    h = Harness(folder, dtype, page_size=8, pages=24)          # 192 tokens of pages: every run reuses the last one's
    ops.reset_kernel_counts()
    whole = h.run(toks)
    assert close(whole, want, clear, dtype), "whole"
    for cuts in ([1], [2], [3, 2, 7, 2, 16, 5], [40, 1, 1, 1], [64, 19]):
        got = h.run(toks, cuts)
        assert close(got, want, clear, dtype), cuts
        if dtype == "float32":
            assert np.array_equal(got, whole), cuts
    if big:        # sizes of the tensor-core kernels: bfloat16 must have taken them, float32 never
        ran = set(ops.kernel_counts())
        fast = {"T": ["attention_prefill_tc_kernel", "attention_prefill_kernel", "attention_decode_kernel"],
                "V": ["attention_prefill_kernel", "masked_attention_mma_kernel"]}[name] + ["gemm_tc_grouped_kernel", "moe_router_kernel"]
        for kernel in fast:
            assert (kernel in ran) == (dtype == "bfloat16"), kernel
        if name == "T":
            assert any(k.startswith("attention_decode_tma_kernel") for k in ran) == (dtype == "bfloat16")
    m = h.storage.manager
    assert all(m.free_pages(g) == h.storage.groups[g].num_pages for g in range(len(h.storage.groups))) and m.free_slots() == 4


@pytest.mark.parametrize("name", ["A", "T"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(tmp_path, dtype, name):
    """Up to three live requests, portions beside single tokens, a request left out of some steps, finished requests'
    pages and slots taken by the next: every row equals the request alone."""
    folder = write_model(CASES[name], str(tmp_path / name), seed=13)
    rng = np.random.default_rng(9)
    lengths = [61, 17, 40, 1, 2, 33, 25]
    reqs = [tokens_of(rng, n, CASES[name]["vocab"]) for n in lengths]
    want = [plain_rows(folder, t, dtype) for t in reqs]
    h = Harness(folder, dtype, page_size=8, pages=20, slots=3)          # 160 tokens: three live requests at most
    alone = [h.run(t) for t in reqs] if dtype == "float32" else None
    waiting, live, done_rows = list(range(len(reqs))), {}, {i: [] for i in range(len(reqs))}
    portions, k, step_no = [2, 5, 1, 9, 3, 14], 0, 0
    while waiting or live:
        while waiting and len(live) < 3 and sum(-(-len(reqs[i]) // 8) for i in live) + -(-len(reqs[waiting[0]]) // 8) <= 20:
            i = waiting.pop(0)
            live[i] = [h.open(), 0]
        entries, who = [], []
        for i, (rid, pos) in list(live.items()):
            if step_no % 4 == 3 and i % 2 == 0 and len(live) > 1:
                continue                                     # left out of this step
            left = len(reqs[i]) - pos
            n = 1 if left <= 6 else min(portions[k % len(portions)], left - 6)      # the last tokens one by one
            k += 1
            entries.append((rid, reqs[i][pos:pos + n], range(n)))
            who.append((i, n))
        step_no += 1
        if not entries:
            continue
        rows, at = h.step(entries), 0
        for i, n in who:
            done_rows[i].append(rows[at:at + n])
            at += n
            live[i][1] += n
            if live[i][1] == len(reqs[i]):
                h.close(live.pop(i)[0])
    got = [np.concatenate(done_rows[i]) for i in range(len(reqs))]
    assert close(np.concatenate(got), np.concatenate([w[0] for w in want]), np.concatenate([w[1] for w in want]), dtype)
    if alone is not None:
        assert all(np.array_equal(a, b) for a, b in zip(got, alone))
    assert h.storage.manager.free_slots() == 3


# ---- a key that stands out: far away, at page borders, at a window's edges; the sink ------------------------------------------
def marker_effect(folder, toks, at):
    """How far the plain model's rows move when the marker at ``at`` is replaced by an ordinary token."""
    want = plain_logits(folder, toks)
    other = list(toks)
    other[at] = ORDINARY
    return want, np.abs(want - plain_logits(folder, other)).max(axis=1) / np.abs(want).max()


#: key and value sizes of the standout models, with the kernels a bfloat16 run must have launched
STANDOUT = {(16, 16): ("attention_prefill_kernel", "attention_decode_kernel"), (64, 64): ("attention_prefill_tc_kernel", "attention_decode_tma_kernel"),
            (32, 16): ("masked_attention_mma_kernel",), (12, 20): ("masked_attention_kernel",)}


@pytest.mark.parametrize("d, dv", sorted(STANDOUT))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_key_among_hundreds_and_at_page_borders(tmp_path, dtype, d, dv):
    """700 tokens behind the marker the penalty on distance is a few tenths of the marker's score in the slight heads and far above it
    in the steep ones; prompts and decoded tokens."""
    from carbon_engine_b200 import ops
    folder = distance_model(str(tmp_path / "far"), d, dv)
    ops.reset_kernel_counts()
    base = [int(t) for t in np.random.default_rng(6).integers(10, 50, 720)]
    h = Harness(folder, dtype, page_size=16, pages=48, max_step_tokens=1024)
    for marker_at in (3, 15, 16, 31, 300):
        toks = list(base)
        toks[marker_at] = MARKER
        want, moved = marker_effect(folder, toks, marker_at)
        assert moved[marker_at:].min() > 0.2 and moved[:marker_at].max() < 1e-12          # the plain model says the far key matters
        assert rel_err(h.run(toks), want) < TOL[dtype], marker_at
        rid = h.open()
        rows = [h.step([(rid, toks[:690], [689])])]
        for p in range(690, 720):
            rows.append(h.step([(rid, toks[p:p + 1], [0])]))
        h.close(rid)
        assert rel_err(np.concatenate(rows), want[689:]) < TOL[dtype], marker_at
    if dtype == "bfloat16":
        for kernel in STANDOUT[(d, dv)]:
            assert any(k.startswith(kernel) for k in ops.kernel_counts()), kernel


@pytest.mark.parametrize("d", [16, 64])
@pytest.mark.parametrize("window", [1, 2, 16, 37, 64, 65, 130])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_just_inside_and_just_outside_the_window(tmp_path, dtype, window, d):
    """The row window - 1 tokens after the marker still sees it, the next one does not; in whole prompts, in portions cut around the
    edge and in decoding, with pages given back as the window passes."""
    folder = window_model(str(tmp_path / f"w{window}"), window, d=d)
    rng = np.random.default_rng(window)
    h = Harness(folder, dtype, page_size=8, pages=64)
    for marker_at in (0, 7, 8, 21, 275):
        n = marker_at + window + 6
        toks = [int(t) for t in rng.integers(10, 50, n)]
        toks[marker_at] = MARKER
        want, moved = marker_effect(folder, toks, marker_at)
        inside, outside = marker_at + window - 1, marker_at + window
        assert moved[marker_at:outside].min() > 0.2 and moved[outside:].max() < 1e-12
        whole = h.run(toks)
        assert rel_err(whole, want) < TOL[dtype], (marker_at, "whole")
        start = max(1, marker_at)
        for cuts in ([2], [max(1, inside), 1], [max(1, outside), 2], [marker_at + 1, 3], [start] + [1] * (n - start)):
            got = h.run(toks, cuts)
            assert rel_err(got, want) < TOL[dtype], (marker_at, cuts[:2])
            if dtype == "float32":
                assert np.array_equal(got, whole)


@pytest.mark.parametrize("d", [16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_takes_its_share_of_every_head(tmp_path, dtype, d):
    """A sink about as large as the marker's score takes much of the marker's weight in two heads and leaves the others alone; a model
    that left it out, scaled it or counted it per key would differ visibly."""
    folder = window_model(str(tmp_path / "sink"), 120, d=d, sink=[26.0, -3.0, 25.0, -20.0])
    no_sink = window_model(str(tmp_path / "none"), 120, d=d, sink=[-30.0] * 4)
    toks = [int(t) for t in np.random.default_rng(2).integers(10, 50, 200)]
    toks[90] = MARKER
    want = plain_logits(folder, toks)
    assert rel_err(plain_logits(no_sink, toks), want) > 0.1            # the plain model itself: the sink matters
    h = Harness(folder, dtype, page_size=8, pages=32)
    whole = h.run(toks)
    assert rel_err(whole, want) < TOL[dtype]
    for cuts in ([1], [2], [150, 3, 1]):
        got = h.run(toks, cuts)
        assert rel_err(got, want) < TOL[dtype], cuts
        if dtype == "float32":
            assert np.array_equal(got, whole)


# ---- the states ---------------------------------------------------------------------------------------------------------
def test_long_decoding_keeps_the_state(tmp_path):
    """300 tokens one by one after a short prompt, in float32: the recurrent states, the convolutions' kept rows and the
    pages must carry every token (bit for bit the rows of the whole prompt)."""
    for name in ("A", "C"):
        folder = write_model(CASES[name], str(tmp_path / name), seed=2)
        toks = tokens_of(np.random.default_rng(8), 310, CASES[name]["vocab"])
        want = plain_logits(folder, toks)
        h = Harness(folder, "float32", page_size=8, pages=48)
        whole = h.run(toks)
        got = h.run(toks, [10] + [1] * 300)
        assert rel_err(got, want) < TOL["float32"] and np.array_equal(got, whole)


def test_an_early_token_reaches_far_through_the_state(tmp_path):
    """With decays close to 1 a token still counts 400 tokens later, long after the attention's window: the plain model says so, and
    the engine's decoded rows agree with it."""
    raw = config([pair(window=5, r_heads=2, r_kv=1, r_dim=24, r_vdim=16, conv=3)], alpha=0.5)

    def change(t):
        t["l0.mix.right.A_log"] = torch.tensor([-7.0, -8.0])
        t["l0.mix.right.b"] = (t["l0.mix.right.b"].float() * 4).to(t["l0.mix.right.b"].dtype)
    folder = write_model(raw, str(tmp_path / "far"), seed=4, change=change)
    toks = tokens_of(np.random.default_rng(10), 420, raw["vocab"])
    want, moved = marker_effect(folder, toks, 2)
    assert moved[400:].min() > 2e-4
    h = Harness(folder, "float32", page_size=8, pages=64, max_step_tokens=512)
    rid = h.open()
    rows = [h.step([(rid, toks[:395], [394])])] + [h.step([(rid, toks[p:p + 1], [0])]) for p in range(395, 420)]
    h.close(rid)
    assert rel_err(np.concatenate(rows), want[394:]) < 0.1 * moved[400:].min()


def test_first_tokens_of_a_sequence_in_a_reused_slot(tmp_path):
    """A slot and pages that held a longer request: the next request's first tokens must start from nothing (zero states, no kept
    convolution inputs, no keys, temperature 1), also when it is shorter than the convolution."""
    for name in ("A", "B"):
        folder = write_model(CASES[name], str(tmp_path / name), seed=5)
        rng = np.random.default_rng(12)
        h = Harness(folder, "float32", page_size=8, pages=12, slots=1, poison=False)
        h.run(tokens_of(rng, 90, CASES[name]["vocab"]))
        for n in (1, 2, 3, 9):
            toks = tokens_of(rng, n, CASES[name]["vocab"])
            want = plain_logits(folder, toks)
            assert rel_err(h.run(toks), want) < TOL["float32"]
            assert rel_err(h.run(toks, [1]), want) < TOL["float32"]


# ---- through the entry point -------------------------------------------------------------------------
@pytest.mark.parametrize("name, graphs", [("A", False), ("A", True), ("B", True)])
def test_greedy_generation_through_the_engine(tmp_path, name, graphs):
    from carbon_engine_b200 import Engine, SamplingParams
    folder = write_model(CASES[name], str(tmp_path / name), seed=17)
    cfg, w = plain.read_model(folder)
    rng = np.random.default_rng(2)
    prompts = [tokens_of(rng, n, cfg["vocab"]) for n in (23, 5, 41)]
    eng = Engine(folder, dtype="float32", page_size=8, max_running_requests=3, max_prefill_tokens=16, kv_tokens=256,
                 cuda_graphs=graphs)
    assert eng.cuda_graphs == graphs
    outs = eng.generate(prompts, SamplingParams(max_tokens=12, ignore_eos=True))
    for prompt, out in zip(prompts, outs):
        assert len(out.token_ids) == 12 and out.finish_reason == "length"
        toks = list(prompt)
        for t in out.token_ids:
            row = plain.forward(cfg, w, toks)[-1]
            assert t == int(row.argmax()) or float(row.max() - row[t]) < 4e-4 * float(row.abs().max())
            toks.append(t)
    eng.storage.manager.check()


def test_decode_steps_as_graphs_give_the_eager_bits_in_bfloat16(tmp_path):
    """The tensor-core sizes with a window, a penalty and mixtures: a step replayed as a CUDA graph is the eager step."""
    from carbon_engine_b200 import Engine, SamplingParams
    folder = write_model(CASES["T"], str(tmp_path / "T"), seed=19)
    rng = np.random.default_rng(4)
    prompts = [tokens_of(rng, n, CASES["T"]["vocab"]) for n in (70, 33)]
    outs = []
    for graphs in (False, True):
        eng = Engine(folder, dtype="bfloat16", page_size=16, max_running_requests=2, max_prefill_tokens=64, kv_tokens=512, cuda_graphs=graphs)
        outs.append([o.token_ids for o in eng.generate(prompts, SamplingParams(max_tokens=24, ignore_eos=True))])
    assert outs[0] == outs[1]


def test_trace_replay_program_on_a_lanirax_folder(tmp_path):
    import json, subprocess, sys
    from helpers import ROOT
    folder = write_model(CASES["A"], str(tmp_path / "A"), seed=1)
    toks = tokens_of(np.random.default_rng(3), 40, CASES["A"]["vocab"])
    want = plain_logits(folder, toks)
    out = str(tmp_path / "out")
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:25], "want": [0, 24]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[25:27], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[27:], "want": [12]}, {"id": "b", "tokens": toks[:3], "want": [2]}],
              "end": ["a", "b"]}]
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                           "--out", out, "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    got0 = np.fromfile(os.path.join(out, "0.f32"), dtype="<f4").reshape(2, -1)
    got2 = np.fromfile(os.path.join(out, "2.f32"), dtype="<f4").reshape(2, -1)
    assert not os.path.exists(os.path.join(out, "1.f32"))
    assert rel_err(got0, want[[0, 24]]) < 2e-4 and rel_err(got2, want[[39, 2]]) < 2e-4


def test_command_line_writes_and_generates_a_lanirax_model(tmp_path):
    """``tiny-model --arch lanirax`` then ``generate``: the printed ids are the plain implementation's greedy ones."""
    import ast, re, subprocess, sys
    from helpers import ROOT
    carbon = [sys.executable, os.path.join(ROOT, "bin", "carbon")]
    out = str(tmp_path / "tiny")
    p = subprocess.run(carbon + ["tiny-model", "--arch", "lanirax", "--out", out, "--layers", "5", "--hidden", "48", "--heads", "3",
                                 "--kv-heads", "1", "--head-dim", "16", "--vocab", "120", "--seed", "9", "--shared-from", "4", "--experts", "6",
                                 "--top-experts", "3", "--mask-size", "7", "--max-positions", "256"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0 and "wrote" in p.stdout, p.stderr[-2000:]
    cfg, w = plain.read_model(out)
    assert cfg["architecture"] == "Lanirax" and len(cfg["layers"]) == 5 and cfg["layers"][4]["weights_of"] == 0
    assert cfg["layers"][0]["mixer"]["left"]["mask"]["size"] == 7 and cfg["layers"][1]["mlp"]["router"] == {"experts": 6, "top": 3}
    prompt = tokens_of(np.random.default_rng(5), 17, 120)
    p = subprocess.run(carbon + ["generate", "--model", out, "--prompt-ids", ",".join(map(str, prompt)), "--max-tokens", "8",
                                 "--ignore-eos", "--print-ids", "--dtype", "f32", "--kv-tokens", "256", "--page-size", "16"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    ids = [ast.literal_eval(m) for m in re.findall(r"output_ids: (\[[^\]]*\])", p.stderr)][0]
    toks = list(prompt)
    for t in ids:
        row = plain.forward(cfg, w, toks)[-1]
        assert t == int(row.argmax()) or float(row.max() - row[t]) < 4e-4 * float(row.abs().max())
        toks.append(t)
    assert len(ids) == 8
