"""Each mechanism of the Vulanex blocks alone: the ops of pie_b200.ops.{stream_conv,delta,grouped} against the plain functions in
vulanex_oracle.py, on the CPU path and on the kernels."""
import math

import numpy as np
import pytest
import torch
import vulanex_oracle as oracle

from pie_b200 import ops
from pie_b200.driver.recurrent import RecurrentInputs
from pie_b200.models.block_spec import EVERYTHING, DeltaRuleSpec, PairSpec, PlainAttentionSpec, RotarySpec
from pie_b200.models.nukelix import _YARN, _scaling
from pie_b200.ops import delta, grouped, stream_conv as conv

F32, BF16 = torch.float32, torch.bfloat16
PATHS = [pytest.param(("cpu", F32), id="cpu"), pytest.param(("cuda", F32), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", BF16), id="cuda-bf16", marks=pytest.mark.gpu)]


def rnd(*shape, seed=0, dtype=F32, std=1.0):
    """Values that are exact in `dtype`, on the CPU in 32-bit."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype).float()


def close(got, ref, dtype, f32=2e-5, bf16=8e-3):
    got, ref = got.float().cpu(), ref.float()
    err = float((got - ref).abs().max()) / max(1e-6, float(ref.abs().max()))
    assert err <= (f32 if dtype == F32 else bf16), err


def recurrent(qo, slots, reset, dev, **kw):
    t = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)
    req = np.repeat(np.arange(len(qo) - 1), np.diff(qo)).tolist()
    return RecurrentInputs(t(qo), t(req), t(slots), t(reset), list(qo), list(slots), list(reset), None, None, {}, **kw)


def padded(parts, dev, dt):
    """The parts side by side as one projection, each on a multiple of 8 columns; their column ranges."""
    cols, at = [], 0
    wide = torch.zeros(parts[0].shape[0], sum(-(-p.shape[1] // 8) * 8 for p in parts))
    for p in parts:
        wide[:, at:at + p.shape[1]] = p
        cols.append((at, p.shape[1]))
        at += -(-p.shape[1] // 8) * 8
    wide = wide.to(dev, dt)
    return [wide[:, a:a + n] for a, n in cols]


# ------------------------------------------------------------------ embedding
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("pair", [(61, 7, 5), (1, 3, 2), (1000003, 999983, 1000000)])
def test_rows_of_token_pairs(path, pair):
    """Sequences in ragged cuts, the token before kept in their slots; products of ids and factors past 32 bits."""
    dev, dt = path
    vocab, w, ld = 70000, 20, 24
    table, pairs = rnd(vocab, w, dtype=dt), rnd(pair[0] + 1, w, seed=1, dtype=dt)
    toks = {r: torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(n)).tolist() for r, n in enumerate((9, 4, 1, 12))}
    toks[1] = [vocab - 1] * 4
    want = {r: oracle.embedding(t, table, pairs, pair[1], pair[2], pair[0]) for r, t in toks.items()}
    state = torch.full((5, 8), float("nan"), device=dev)
    at = dict.fromkeys(toks, 0)
    for fire in ([(0, 3), (1, 1), (2, 1)], [(1, 1), (0, 1)], [(3, 12), (0, 2), (1, 2)], [(0, 3)]):
        qo = np.concatenate([[0], np.cumsum([k for _, k in fire])]).tolist()
        rs = recurrent(qo, [r + 1 for r, _ in fire], [int(at[r] == 0) for r, _ in fire], dev, linear_state=state, token_at=5)
        ids = [x for r, k in fire for x in toks[r][at[r]:at[r] + k]]
        got = conv.pair_embed(torch.tensor(ids, dtype=torch.int32, device=dev), table.to(dev, dt), pairs.to(dev, dt), PairSpec(*pair), ld, rs)
        assert got.dtype == F32 and not got[:, w:].any()
        close(got[:, :w], torch.cat([want[r][at[r]:at[r] + k] for r, k in fire]), F32)
        for r, k in fire:
            at[r] += k
    assert state[:, [0, 1, 2, 3, 4, 6, 7]].isnan().all() and state[0].isnan().all()


# ------------------------------------------------------------------ layer norm and convolution
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("width", [48, 51])
def test_norm_and_convolution_in_portions(path, taps, width):
    """Requests in ragged cuts, some shorter than the convolution's reach; a history that is not the sequence's own must not leak in."""
    dev, dt = path
    lens = [40, 9, 1, 30]
    x = {r: rnd(n, width, seed=r, std=2) + 3 for r, n in enumerate(lens)}
    w, b, c = rnd(width, seed=10), rnd(width, seed=11), rnd(width, taps, seed=12)
    want = {r: oracle.input_convolution(oracle.layer_norm(v, w, b, 1e-3), c) for r, v in x.items()}
    factors = c.t().contiguous()
    factors[-1] += 1
    ld = -(-width // 8) * 8
    cache = torch.full((5, (taps - 1) * width + 8), float("nan"), device=dev)
    history = cache[:, 4:4 + (taps - 1) * width] if taps > 1 else None
    d = lambda t: t.to(dev)
    at = dict.fromkeys(x, 0)
    for fire in ([(0, 5), (1, 2)], [(0, 1), (1, 1), (2, 1), (3, 2)], [(3, 1), (0, 20), (1, 6)], [(0, 2), (3, 3)], [(0, 12), (3, 24)]):
        n = sum(k for _, k in fire)
        qo = np.concatenate([[0], np.cumsum([k for _, k in fire])]).tolist()
        rs = recurrent(qo, [r + 1 for r, _ in fire], [int(at[r] == 0) for r, _ in fire], dev)
        rs.conv_stage = torch.full((len(fire), max(1, (taps - 1) * width)), float("nan"), device=dev)
        rows = torch.zeros(n, ld)
        rows[:, :width] = torch.cat([x[r][at[r]:at[r] + k] for r, k in fire])
        same, h = conv.conv_norm(d(rows), width, 1e-3, (), d(w), d(b), d(factors), history, rs, dt)
        assert torch.equal(same.cpu(), rows) and h.dtype == dt and not h[:, width:].any()
        close(h[:, :width], torch.cat([want[r][at[r]:at[r] + k] for r, k in fire]), dt)
        for r, k in fire:
            at[r] += k
    assert all(at[r] == n for r, n in enumerate(lens)) and cache[0].isnan().all() and cache[:, :4].isnan().all()
    if taps > 1:
        last = oracle.layer_norm(x[0], w, b, 1e-3)[-(taps - 1):]
        close(history[1].view(taps - 1, width), last, F32)


@pytest.mark.parametrize("path", PATHS[1:])
@pytest.mark.parametrize("taps", [3, 4, 6])
@pytest.mark.parametrize("pending", [0, 1, 2])
def test_norm_and_convolution_of_many_rows(path, taps, pending):
    """Portions around the rows that a block takes, sublayer outputs that join the stream on the way."""
    dev, dt = path
    width, lens, ld = 320, [700, 1, 2, 15, 16, 17, 33, 400], 328
    n = sum(lens)
    x, ys = rnd(n, width, std=3), [rnd(n, width, seed=20 + i, dtype=dt) for i in range(pending)]
    gains = [rnd(width, seed=30 + i) for i in range(pending)]
    w, b, c = rnd(width, seed=1), rnd(width, seed=2), rnd(width, taps, seed=3, std=0.5)
    total = x + sum(oracle.rms(y, 1e-5) * g for y, g in zip(ys, gains))
    qo = np.concatenate([[0], np.cumsum(lens)]).tolist()
    normed = [oracle.layer_norm(total[a:e], w, b, 1e-5) for a, e in zip(qo, qo[1:])]
    factors = c.t().contiguous()
    factors[-1] += 1
    wide = lambda t: torch.nn.functional.pad(t, (0, ld - width))
    rs = recurrent(qo, list(range(1, len(lens) + 1)), [1] * len(lens), dev)
    rs.conv_stage = torch.full((len(lens), (taps - 1) * width), float("nan"), device=dev)
    history = torch.full((len(lens) + 1, (taps - 1) * width), float("nan"), device=dev)
    out, h = conv.conv_norm(wide(x).to(dev), width, 1e-5, tuple((wide(y).to(dev, dt), g.to(dev)) for y, g in zip(ys, gains)), w.to(dev), b.to(dev),
                            factors.to(dev), history, rs, dt)
    close(out[:, :width], total, F32)
    assert not out[:, width:].any() and not h[:, width:].any()
    close(h[:, :width], torch.cat([oracle.input_convolution(y, c) for y in normed]), dt)
    for r, y in enumerate(normed):
        close(history[r + 1].view(taps - 1, width), torch.cat([torch.zeros(taps - 1, width), y])[-(taps - 1):], F32)


@pytest.mark.parametrize("path", PATHS)
def test_norm_of_rows_far_from_zero(path):
    """A mean a thousand times the deviation; no convolution; sublayer outputs alone."""
    dev, dt = path
    x, w, b = 1000 + rnd(6, 64), rnd(64, seed=1), rnd(64, seed=2)
    _, h = conv.conv_norm(x.to(dev), 64, 1e-5, w=w.to(dev), b=b.to(dev), dtype=dt)
    close(h, oracle.layer_norm(x.double(), w.double(), b.double(), 1e-5), dt, f32=2e-4)
    y, g = rnd(6, 64, seed=3, dtype=dt), rnd(64, seed=4)
    out, none = conv.conv_norm(x.to(dev), 64, 1e-5, ((y.to(dev, dt), g.to(dev)),))
    assert none is None
    close(out, x + oracle.rms(y, 1e-5) * g, F32)


# ------------------------------------------------------------------ attention
#      heads, kv, dim, vdim, rotated, window, block, sink;  rotated 0: values are keys, factor on the query
ATT = {"g3": (6, 2, 40, 24, 24, 37, 5, True), "g1": (3, 3, 64, 64, 64, 64, 16, True), "g4": (8, 2, 128, 128, 64, 129, 4, True),
       "g8": (8, 1, 72, 100, 20, 70, 33, True), "d256": (4, 2, 136, 200, 136, 50, 17, True), "any": (20, 1, 24, 24, 8, 60, 9, True),
       "huge": (2, 1, 264, 300, 2, 33, 3, True), "one": (2, 2, 8, 16, 8, 1, 1, True), "no sink": (16, 1, 128, 96, 128, 20, 2, False),
       "own": (6, 3, 64, 64, 0, EVERYTHING, 0, False), "own 128": (8, 2, 128, 128, 0, EVERYTHING, 0, False),
       "own any": (20, 1, 40, 40, 0, EVERYTHING, 0, False), "own 256": (4, 1, 200, 200, 0, EVERYTHING, 0, False)}


def att_spec(name):
    h, kv, d, e, rot, w, pool, sink = ATT[name]
    if not rot:
        return PlainAttentionSpec(h, kv, d, e, 1.2 * d ** -0.5, q_temp=(0.3, 11), shared_kv=True)
    s = {"scaling": {"factor": 3.0, "original": 50, "fast": 6.0, "slow": 1.0}}
    return PlainAttentionSpec(h, kv, d, e, 1.2 * d ** -0.5, RotarySpec(rot, 200.0, False, _scaling(s, "yarn", _YARN)), True, window=w, pool=pool,
                              sink=sink)


@pytest.mark.parametrize("dims,base,s", [(32, 700.0, (4.0, 64, 8.0, 1.0)), (64, 1e6, (2.0, 700, 32.0, 1.0)), (2, 9.0, (2.0, 30, 3.0, 1.0)),
                                         (20, 1e6, (1.0, 100, 2.0, 1.5)), (8, 30.0, (3.0, 7, 32.0, 20.0))])
def test_frequencies(dims, base, s):
    rot = {"dims": dims, "base": base, "scaling": dict(zip(("factor", "original", "fast", "slow"), s))}
    r = RotarySpec(dims, base, False, _scaling(rot, "yarn", _YARN))
    f, factor = oracle.stretched_frequencies(rot)
    assert torch.allclose(r.frequencies(), f.float(), rtol=1e-6, atol=0) and r.factor == pytest.approx(factor)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "g8", "d256", "one", "huge", "own", "own any"])
def test_rows_normed_per_head_rotated_or_scaled(path, name):
    dev, dt = path
    spec, n, page, eps = att_spec(name), 9, 16, 1e-3
    nq, nk = spec.heads * spec.dim, spec.kv_heads * spec.dim
    parts = [rnd(n, nq, dtype=dt, std=3), rnd(n, nk, seed=1, dtype=dt, std=0.1)] + \
        ([] if spec.shared_kv else [rnd(n, spec.kv_heads * spec.vdim, seed=2, dtype=dt)])
    gq, gk = rnd(spec.dim, seed=6), rnd(spec.dim, seed=7)
    pos = [0, 1, 2, 5, 63, 64, 1000, 4095, 10]
    slots = torch.tensor([4, 9, 0, 31, 17, 2, -1, 30, 16], dtype=torch.int32)
    cache = torch.full((3, spec.planes, spec.kv_heads, page, spec.head_dim), 0.0 if dev == "cpu" else 7.0, dtype=dt, device=dev)
    cols = padded(parts, dev, dt)
    lw = {"q_gain": gq.to(dev), "k_gain": gk.to(dev), "rope": spec.rot.frequencies(dev)} if spec.rot else {}
    got = grouped.head_rows(cols[0], cols[1], cols[2] if len(cols) > 2 else None, lw, torch.tensor(pos, dtype=torch.int32, device=dev),
                            slots.to(dev), cache, spec, eps)
    heads = lambda x: x.view(n, -1, spec.dim)
    q, k = heads(parts[0]), heads(parts[1])
    v = k if spec.shared_kv else parts[2].view(n, spec.kv_heads, spec.vdim)
    if spec.rot:
        s = {k_: spec.rot.scaling[v_] for k_, v_ in _YARN.items()}
        f, factor = oracle.stretched_frequencies({"dims": spec.rot.dims, "base": spec.rot.base, "scaling": s})
        q, k = (oracle.rotated(oracle.rms(x, eps) * g, f, factor, pos) for x, g in ((q, gq), (k, gk)))
    else:
        q = q * oracle.query_factor(torch.tensor(pos, dtype=F32), *spec.q_temp)[:, None, None]
    rows = got.view(n, spec.kv_heads, spec.group_pad, spec.head_dim).float().cpu()
    close(rows[:, :, :spec.group, :spec.dim].reshape(n, spec.heads, spec.dim), q, dt, f32=3e-4)
    assert not rows[:, :, spec.group:].any() and not rows[..., spec.dim:].any()
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            at = cache[s // page, :, :, s % page].float().cpu()
            close(at[0, :, :spec.dim], k[i], dt, f32=3e-4)
            close(at[-1, :, :spec.vdim], v[i], dt)
            assert not at[0, :, spec.dim:].any() and not at[-1, :, spec.vdim:].any()


def attention_case(spec, kv_lens, qlens, page, dev, dt, seed=0):
    """Rows in shuffled pages. For some queries there are keys far more alike than the rest: on both sides of the window's edge,
    at a page's border, and whole blocks of them, the last one seen and the first one that is not yet."""
    total, D, pool = sum(-(-n // page) for n in kv_lens), spec.head_dim, spec.pool
    order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.zeros(total + 1, spec.planes, spec.kv_heads, page, D)
    qs, ks, vs, tables = [], [], [], []
    u = rnd(spec.dim, seed=99, dtype=dt)
    for i, (n, ql) in enumerate(zip(kv_lens, qlens)):
        q = rnd(ql, spec.heads, spec.dim, seed=seed + 10 * i + 1, dtype=dt)
        k, v = rnd(n, spec.kv_heads, spec.dim, seed=seed + 10 * i + 2, dtype=dt), rnd(n, spec.kv_heads, spec.vdim, seed=seed + 10 * i + 3, dtype=dt)
        for t in (0, ql // 2, ql - 1):
            pos = n - ql + t
            q[t] += 0.6 * u
            stand_out = [0, pos, pos // page * page]
            if spec.window != EVERYTHING:
                seen = max(0, pos - spec.window + 1) // pool
                stand_out += [pos - spec.window + 1, pos - spec.window] + (list(range((seen - 1) * pool, (seen + 1) * pool)) if i % 2 else [])
            for j in stand_out:
                if 0 <= j < n:
                    k[j] = (1.5 * u).to(dt).float()
        q = q.to(dt).float()
        if spec.shared_kv:
            v = k
        table = [order.pop() for _ in range(-(-n // page))]
        for j in range(n):
            cache[table[j // page], 0, :, j % page, :spec.dim] = k[j]
            cache[table[j // page], -1, :, j % page, :spec.vdim] = v[j]
        qs.append(q), ks.append(k), vs.append(v), tables.append(table)
    indptr = np.concatenate([[0], np.cumsum([len(t) for t in tables])]).astype(np.int32)
    batch = ops.AttnBatch(np.concatenate([[0], np.cumsum(qlens)]).astype(np.int32), indptr, np.concatenate(tables).astype(np.int32),
                          np.asarray(kv_lens, np.int32), None, -1)
    rows = torch.zeros(sum(qlens), spec.kv_heads, spec.group_pad, D)
    rows[:, :, :spec.group, :spec.dim] = torch.cat(qs).view(-1, spec.kv_heads, spec.group, spec.dim)
    means = None
    if pool:                                    # places of blocks that do not exist yet, or whose page was another's, hold anything
        means = torch.full((total + 1, 2, spec.kv_heads, -(-page // pool), D), 50.0)
        for n, k, v, table in zip(kv_lens, ks, vs, tables):
            for blk in range(n // pool):
                at = ((blk + 1) * pool - 1) // page
                row = blk - at * page // pool
                means[table[at], :, :, row] = 0
                means[table[at], 0, :, row, :spec.dim] = k[blk * pool:(blk + 1) * pool].mean(0)
                means[table[at], 1, :, row, :spec.vdim] = v[blk * pool:(blk + 1) * pool].mean(0)
        means = means.to(dev, dt)
    return qs, ks, vs, batch, rows.view(sum(qlens), -1, D).to(dev, dt), cache.to(dev, dt), means


def learned(spec):
    return rnd(spec.heads, seed=55) if spec.sink else torch.full((spec.heads,), -1e30)


def plain_attention(spec, qs, ks, vs, dt, masks=None):
    out = []
    for i, (q, k, v) in enumerate(zip(qs, ks, vs)):
        n, ql, pool = k.shape[0], q.shape[0], spec.pool or k.shape[0] + 1
        keys = torch.cat([k, oracle.block_means(k, pool).to(dt).float()]).repeat_interleave(spec.group, 1)
        values = torch.cat([v, oracle.block_means(v, pool).to(dt).float()]).repeat_interleave(spec.group, 1)
        see, blocks = oracle.seen_tokens(n, spec.window)[n - ql:], oracle.seen_blocks(n, spec.window, pool)[n - ql:]
        if masks is not None:
            see, blocks = see & masks[i], blocks & masks[i][:, :n // pool * pool].reshape(ql, -1, pool).all(-1)
        p = oracle.weights_with_sink(torch.einsum("ihd,jhd->hij", q, keys) * spec.scale, torch.cat([see, blocks], 1), learned(spec))
        out.append(torch.einsum("hij,jhd->ihd", p, values))
    return torch.cat(out)


def spread(out, spec):
    n = out.shape[0]
    assert not out.view(n, spec.kv_heads, spec.group_pad, -1)[..., spec.vdim:].any()
    return out.view(n, spec.kv_heads, spec.group_pad, -1)[:, :, :spec.group, :spec.vdim].reshape(n, spec.heads, spec.vdim)


def sinks(spec, dev):
    if not spec.sink:
        return None
    s = torch.zeros(spec.kv_heads, spec.group_pad)
    s[:, :spec.group] = learned(spec).view(spec.kv_heads, spec.group)
    return s.flatten().to(dev), (s.flatten() / math.log(2)).to(dev)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("page", [16, 32])
def test_attention_of_portions(path, name, page):
    """Prompts and portions of prompts: around the edges of the window and of the blocks, over page and key block borders."""
    dev, dt = path
    spec = att_spec(name)
    kv_lens, qlens = ([47, 1, 30, 64, 90], [47, 1, 2, 20, 3]) if dev == "cpu" else ([230, 1, 130, 64, 390, 700], [230, 1, 2, 20, 100, 5])
    qs, ks, vs, batch, q, cache, means = attention_case(spec, kv_lens, qlens, page, dev, dt)
    rs = recurrent(batch.qo_indptr.tolist(), list(range(len(qlens))), [0] * len(qlens), dev)
    plan = batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, page, dev)
        plan.host = batch
    got = grouped.laid_attention(q, cache, means, plan, rs, torch.zeros(q.shape[0], dtype=torch.int32, device=dev), spec, sinks(spec, dev))
    close(spread(got, spec), plain_attention(spec, qs, ks, vs, dt), dt, bf16=1.2e-2)
    if dev != "cpu":
        ops.check_kernel_status()


@pytest.mark.parametrize("path", PATHS[1:])
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("chunk", [32, 256])
def test_attention_of_decode_steps(path, name, chunk):
    """Contexts of many lengths in one decode step, split over more or fewer work items."""
    dev, dt = path
    spec = att_spec(name)
    w, pool = min(spec.window, 150), spec.pool or 16
    kv_lens = sorted({1, 2, 15, 16, 17, max(1, w - 1), w, w + 1, w + pool - 1, w + pool, w + 15 * pool, w + 16 * pool, w + 17 * pool, 200, 333, 900})
    qs, ks, vs, batch, q, cache, means = attention_case(spec, kv_lens, [1] * len(kv_lens), 16, dev, dt)
    r, sms = len(kv_lens), ops.num_sms()
    ir, st, en, indptr = ops.plan_decode_items(np.asarray(kv_lens), spec.kv_heads, 2 * sms, r + 16 * sms, min_chunk=chunk)
    t = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    scratch = torch.full((ops.decode_scratch_floats(r + 16 * sms, q.shape[1], spec.head_dim),), float("nan"), device=dev)
    plan = ops.DecodePlan(t(batch.page_indices), t(batch.kv_page_indptr), t(ir), t(st), t(en), t(indptr), t([len(ir)]), scratch,
                          r + 16 * sms, r, 2 * sms, 16, -1, kv_lens=t(kv_lens))
    rs = recurrent(list(range(r + 1)), list(range(r)), [0] * r, dev)
    got = grouped.laid_attention(q, cache, means, plan, rs, torch.zeros(r, dtype=torch.int32, device=dev), spec, sinks(spec, dev))
    close(spread(got, spec), plain_attention(spec, qs, ks, vs, dt), dt, bf16=1.2e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "d256", "own"])
def test_attention_under_a_custom_mask(path, name):
    """A mask chooses among the visible keys; a mean counts where the mask shows all its tokens."""
    dev, dt = path
    spec, n, ql = att_spec(name), 115, 30
    qs, ks, vs, batch, q, cache, means = attention_case(spec, [n], [ql], 16, dev, dt)
    mask = torch.rand(ql, n // 23, generator=torch.Generator().manual_seed(3)).repeat_interleave(23, 1) < 0.6
    mask &= torch.arange(n)[None] <= torch.arange(n - ql, n)[:, None]
    mask[:, n - ql:] |= torch.eye(ql, dtype=torch.bool)
    batch.masks, plan = [mask.numpy()], batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, 16, dev)
        plan.host = batch
        plan.mask_bits, plan.mask_word_indptr = ops.pack_masks([mask.numpy()], [n], dev)
    got = grouped.laid_attention(q, cache, means, plan, recurrent([0, ql], [0], [0], dev), torch.zeros(ql, dtype=torch.int32, device=dev), spec,
                                 sinks(spec, dev))
    close(spread(got, spec), plain_attention(spec, qs, ks, vs, dt, [mask]), dt, bf16=1.2e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("page", [16, 32])
@pytest.mark.parametrize("pool", [1, 5, 16, 24, 50])
def test_means_of_completed_blocks(path, page, pool):
    """Portions that complete no block, one or several, blocks that straddle pages or are longer than one; other places stay."""
    dev, dt = path
    spec = PlainAttentionSpec(2, 2, 16, 16, 1.0, window=3, pool=pool)
    kv_lens, qlens = [47, 50, 1, 100, 96], [47, 1, 1, 30, 24]
    _, ks, vs, batch, q, cache, means = attention_case(spec, kv_lens, qlens, page, dev, dt)
    got = torch.full_like(means, 9.0)
    slots = torch.zeros(sum(qlens), dtype=torch.int32, device=dev)
    slots[47] = -1                                      # the second request is padding
    rs = recurrent(batch.qo_indptr.tolist(), list(range(5)), [0] * 5, dev)
    plan = batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, page, dev)
    grouped.pool_rows(cache, got, plan, rs, slots, spec)
    want = torch.full_like(means, 9.0)
    for r, (n, ql) in enumerate(zip(kv_lens, qlens)):
        for blk in range((n - ql) // pool, n // pool):
            at = ((blk + 1) * pool - 1) // page
            pg = batch.page_indices[batch.kv_page_indptr[r] + at]
            if r != 1:
                want[pg, :, :, blk - at * page // pool] = means[pg, :, :, blk - at * page // pool]
    close(got, want.cpu(), dt, bf16=8e-3)


# ------------------------------------------------------------------ delta rule
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("n,channels,rank", [(3, 10, 1), (70, 130, 24), (1, 64, 16), (130, 72, 300), (1500, 200, 40)])
def test_bounded_decays(path, n, channels, rank):
    dev, dt = path
    x, w2, w0 = rnd(n, rank, dtype=dt, std=2), rnd(channels, rank, seed=1, dtype=dt, std=2 * rank ** -0.5), rnd(channels, seed=2, dtype=dt, std=3)
    w = {"w1": torch.eye(rank), "w2": w2, "w0": w0}
    got = delta.bounded_decay_logs(padded([rnd(n, 8), x], dev, dt)[1], w2.to(dev, dt), w0.to(dev, dt), math.exp(-0.5))
    assert got.dtype == F32
    close(torch.exp2(got), oracle.decays(x, w), F32, f32=2e-5)


DELTA = [(1, 1), (3, 7), (2, 32), (2, 40), (1, 64), (2, 100), (2, 128), (1, 136), (1, 260)]


def delta_case(n, h, d, dt, kind):
    x = [rnd(n, h * d, seed=s, dtype=dt) for s in range(4)]
    b = rnd(h * d, seed=5)
    decay = oracle.sigmoid(rnd(n, h * d, seed=6, std=2)) * -math.exp(-0.5)
    if kind == "fleeting":                      # decays at their bound, everything removed that is asked for
        decay, b = torch.full_like(decay, -math.exp(-0.5)), b + 30
    if kind == "lasting":
        decay, b = decay * 1e-3, b - 3
    if kind == "silent":                        # keys next to nothing between ordinary ones
        x[1][::3] *= 1e-4
        x[1] = x[1].to(dt).float()
    return x, b, decay


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("h,d", DELTA)
@pytest.mark.parametrize("kind", ["steady", "fleeting", "lasting", "silent"])
def test_delta_rule_in_portions(path, h, d, kind):
    """One sequence in portions of many sizes, whose state lives in one slot."""
    dev, dt = path
    sizes = [1, 2, 1, 3, 10, 23] if dev == "cpu" else [2, 16, 1, 1, 15, 17, 3, 64, 200, 33]
    n = sum(sizes)
    (r, k, v, a), b, decay = delta_case(n, h, d, dt, kind)
    heads = lambda y: y.double().view(n, h, d)
    ref, s = oracle.delta_rule(heads(r), heads(k), heads(v), heads(decay.exp()), oracle.sigmoid(heads(a + b)))
    spec = DeltaRuleSpec(h, d, 4)
    cache = torch.full((3, -(-spec.state_elems // 4) * 4 + 8), float("nan"), device=dev)      # an unset slot must not leak in
    state, at, out = cache[:, 4:4 + spec.state_elems], 0, []
    for size in sizes:
        rs = recurrent([0, size], [1], [1 if at == 0 else 0], dev)
        p = slice(at, at + size)
        cols = padded([y[p] for y in (r, k, v, a)], dev, dt)
        out.append(delta.delta_rule(*cols, b.to(dev), (decay[p] / math.log(2)).to(dev), spec, rs, state, size == 1))
        at += size
    close(torch.cat(out).view(n, h, d), ref, dt, f32=3e-5, bf16=2e-3)
    close(state[1].view(h, d, d), s, dt, f32=3e-5, bf16=2e-3)
    assert not state[0].isfinite().any() and not state[2].isfinite().any() and cache[:, :4].isnan().all()


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("h,d", [(2, 24), (1, 128), (1, 130)])
def test_delta_rule_over_a_ragged_batch(path, h, d):
    """Portions beside single tokens, sequences that go on and that start, a padding request."""
    dev, dt = path
    lens, reset = [5, 1, 40, 17, 1, 3], [0, 0, 1, 0, 1, 0]
    n, qo = sum(lens), np.concatenate([[0], np.cumsum(lens)]).tolist()
    (r, k, v, a), b, decay = delta_case(n, h, d, dt, "steady")
    spec, slots = DeltaRuleSpec(h, d, 4), [3, 0, 5, 1, 2, -1]
    start = rnd(6, spec.state_elems, seed=9)
    state = start.clone().to(dev)
    got = delta.delta_rule(*padded([r, k, v, a], dev, dt), b.to(dev), (decay / math.log(2)).to(dev), spec, recurrent(qo, slots, reset, dev),
                           state, False)
    for i, (p, e) in enumerate(zip(qo[:-2], qo[1:-1])):
        heads = lambda y: y[p:e].double().view(e - p, h, d)
        old = None if reset[i] else start[slots[i]].double().view(h, d, d)
        ref, s = oracle.delta_rule(heads(r), heads(k), heads(v), heads(decay.exp()), oracle.sigmoid(heads(a + b)), old)
        close(got[p:e].view(-1, h, d), ref, dt, f32=3e-5, bf16=2e-3)
        close(state[slots[i]].view(h, d, d), s, dt, f32=3e-5, bf16=2e-3)
    assert torch.equal(state[4].cpu(), start[4])


# ------------------------------------------------------------------ feed-forward
@pytest.mark.gpu
@pytest.mark.parametrize("m,n,k", [(1, 96, 64), (16, 2048, 4096), (64, 4096, 1024), (130, 352, 264), (700, 1024, 512), (2048, 4096, 4096)])
def test_gelu_in_the_epilogue_of_gate_and_up(m, n, k):
    """All forms of the product: whole tiles, swapped operands, K split over the CTAs, CTA pairs."""
    x, w = rnd(m, k, dtype=BF16), rnd(n, k, seed=1, dtype=BF16, std=2 * k ** -0.5)
    got = ops.gemm(x.cuda().bfloat16(), w.cuda().bfloat16(), epilogue=ops.EPI_GEGLU)
    y = (x.cuda().double() @ w.cuda().double().t()).cpu()
    want = oracle.gelu_tanh(y[:, 0::2]) * y[:, 1::2]
    assert got.shape == (m, n // 2)
    close(got, want, BF16, bf16=6e-3)
    ops.check_kernel_status()
