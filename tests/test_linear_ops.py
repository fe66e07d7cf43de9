"""Each mechanism of the Retodra blocks alone: the ops of pie_b200.ops.linear (and the expert, stream and embedding ops they
share with other designs) against the plain functions in retodra_oracle.py, on the CPU path and on the kernels."""
import math

import numpy as np
import pytest
import retodra_oracle as oracle
import torch

from pie_b200 import ops
from pie_b200.driver.recurrent import RecurrentInputs
from pie_b200.models.block_spec import BiasedAttentionSpec, ExpertsSpec, GatedLinearSpec, LightningSpec
from pie_b200.ops import latent as lops, linear as lin, linear_reference as lref

F32, BF16 = torch.float32, torch.bfloat16
PATHS = [pytest.param(("cpu", F32), id="cpu"), pytest.param(("cuda", F32), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", BF16), id="cuda-bf16", marks=pytest.mark.gpu)]
gpu = pytest.mark.gpu


def rnd(*shape, seed=0, dtype=F32, std=1.0):
    """Values that are exact in `dtype`, on the CPU in 32-bit."""
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std).to(dtype).float()


def close(got, ref, dtype, f32=2e-5, bf16=8e-3):
    got, ref = got.float().cpu(), ref.float()
    err = float((got - ref).abs().max()) / max(1e-6, float(ref.abs().max()))
    assert err <= (f32 if dtype == F32 else bf16), err


def recurrent(qo, slots, reset, dev):
    t = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)
    req = np.repeat(np.arange(len(qo) - 1), np.diff(qo)).tolist()
    return RecurrentInputs(t(qo), t(req), t(slots), t(reset), list(qo), list(slots), list(reset), None, None, {})


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


# ------------------------------------------------------------------ linear attention
SHAPES = [(1, 1, 1), (3, 7, 11), (2, 32, 64), (2, 40, 24), (1, 128, 128), (3, 96, 36), (1, 200, 64), (1, 272, 24), (2, 64, 260)]


def channel_case(n, h, d, e, dt, strength, seed=0):
    q, k, v = rnd(n, h * d, seed=seed, dtype=dt), rnd(n, h * d, seed=seed + 1, dtype=dt, std=d ** -0.5), rnd(n, h * e, seed=seed + 2, dtype=dt)
    logs = -torch.rand(n, h * d, generator=torch.Generator().manual_seed(seed + 3)) * strength
    logs[:, ::3] *= 0.01                        # some channels remember for long
    return q, k, v, logs


def plain(q, k, v, a, h, keep=None):
    n = q.shape[0]
    return oracle.decayed_state(q.view(n, h, -1), k.view(n, h, -1), v.view(n, h, -1), a, keep).reshape(n, -1)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("h,d,e", SHAPES)
@pytest.mark.parametrize("kind", ["channel", "steep", "abrupt", "head"])
def test_linear_attention_in_portions(path, h, d, e, kind):
    """One sequence in portions of many sizes, whose state lives in one slot; every form of the decay."""
    dev, dt = path
    n = 40 if dev == "cpu" else 300
    strength = {"channel": 0.1, "steep": 3.0, "abrupt": 40.0, "head": 0.0}[kind]
    q, k, v, logs = channel_case(n, h, d, e, dt, strength)
    decay = torch.tensor([1.0, 0.97, 0.4][:h] + [0.9] * max(0, h - 3))
    silu = kind == "head"
    act = oracle.silu if silu else (lambda x: x)
    a = decay[None, :, None].expand(n, h, d) if silu else logs.view(n, h, d).exp()
    states = []
    ref = plain(act(q) * d ** -0.5, act(k), act(v), a, h, states)
    spec = LightningSpec(h, d, e, decay.tolist()) if silu else GatedLinearSpec(h, d, e, 1.0, 4)
    base = logs if dev == "cpu" else logs * lin.LOG2E
    cache = torch.full((3, spec.state_elems + 8), float("nan"), device=dev)      # an unset slot must not leak in
    state = cache[:, 4:4 + spec.state_elems]
    at, out = 0, []
    sizes = ([1, 2, 1, 3, 10, 23] if dev == "cpu" else [2, 64, 1, 1, 63, 65, 3, 17, 84])
    for i, size in enumerate(sizes):
        rs = recurrent([0, size], [1], [1 if at == 0 else 0], dev)
        qq, kk, vv = padded([x[at:at + size] for x in (q, k, v)], dev, dt)
        out.append(lin.linear_attention(qq, kk, vv, spec, rs, state, size == 1, None if silu else base[at:at + size].to(dev).contiguous(),
                                        decay.to(dev) if silu else None, silu, d ** -0.5).cpu())
        at += size
    limit = 8e-3 if silu else 4e-3                # the activations of a prompt's queries and keys may be rounded
    close(torch.cat(out), ref[:at], dt, bf16=limit)
    close(state[1].cpu().view(h, d, e), states[at - 1], dt, bf16=limit)
    assert not state[0].isfinite().any() and not state[2].isfinite().any()


@pytest.mark.parametrize("path", PATHS)
def test_linear_attention_over_a_ragged_batch(path):
    """Unequal portions in one launch: fresh and continued slots, a padding row, states of their own."""
    dev, dt = path
    h, d, e = 2, 24, 40
    lens = [5, 1, 0, 33, 2] if dev == "cpu" else [70, 1, 0, 200, 2]
    slots, reset = [3, -1, 0, 4, 1], [1, 0, 0, 0, 1]
    qo = np.concatenate([[0], np.cumsum(lens)]).tolist()
    q, k, v, logs = channel_case(qo[-1], h, d, e, dt, 0.3, 7)
    before = rnd(6, h * d * e, seed=9)
    state = before.clone().to(dev)
    base = (logs if dev == "cpu" else logs * lin.LOG2E).to(dev)
    qq, kk, vv = padded([q, k, v], dev, dt)
    rs = recurrent(qo, slots, reset, dev)
    got = lin.linear_attention(qq, kk, vv, GatedLinearSpec(h, d, e, 1.0, 4), rs, state, False, base)
    for r, (a, b) in enumerate(zip(qo, qo[1:])):
        if slots[r] < 0 or a == b:
            continue
        s = torch.zeros(h, d, e) if reset[r] else before[slots[r]].view(h, d, e)
        want = []
        for t in range(a, b):
            s = logs[t].exp().view(h, d, 1) * s + k[t].view(h, d, 1) * v[t].view(h, 1, e)
            want.append((s * q[t].view(h, d, 1)).sum(1).reshape(-1))
        close(got[a:b], torch.stack(want), dt, bf16=4e-3)
        close(state[slots[r]].cpu().view(h, d, e), s, dt, bf16=4e-3)
    for s in (0, 2, 5):
        assert torch.equal(state[s].cpu(), before[s])


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("n,c,rank,tau", [(1, 5, 1, 1.0), (19, 300, 16, 16.0), (8, 64, 33, 3.0)])
def test_channel_decays(path, n, c, rank, tau):
    dev, dt = path
    x, a2, b = rnd(n, rank, dtype=dt, std=3), rnd(c, rank, seed=1, dtype=dt, std=2), rnd(c, seed=2, dtype=dt, std=4)
    (xx,) = padded([x], dev, dt)
    got = lin.decay_logs(xx, a2.to(dev, dt), b.to(dev, dt), tau).cpu() / (1.0 if dev == "cpu" else lin.LOG2E)
    want = oracle.log_sigmoid(x.double() @ a2.double().t() + b.double()) / tau
    assert float((got - want).abs().max()) <= 2e-6 * float(want.abs().max())
    some = want.abs() > 1e-9            # also where the decay is next to none
    assert float(((got - want).abs() / want.abs())[some].max()) < 1e-4


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("heads,kv,vdim,cols", [(6, 2, 24, 144), (5, 1, 33, 165), (4, 4, 8, 32)])
def test_gated_norms(path, heads, kv, vdim, cols):
    dev, dt = path
    n, eps = 7, 1e-3
    spec = BiasedAttentionSpec(heads, kv, 8, vdim, 4, 1.0, 5.0, 9, 8)
    left, right = rnd(n, heads, vdim, dtype=dt), rnd(n, cols, seed=1)
    g1, g2, w = rnd(n, heads * vdim, seed=2, dtype=dt, std=2), rnd(n, cols, seed=3, dtype=dt, std=2), rnd(cols, seed=4, dtype=dt)
    x = torch.full((n, kv, spec.group_pad, spec.head_dim), 9.0)
    x[:, :, :spec.group, :vdim] = left.view(n, kv, spec.group, vdim)
    ga, gb = padded([g1, g2], dev, dt)
    cut = -(-heads * vdim // 8) * 8
    z = torch.full((n, cut + cols + 8), 5.0, dtype=dt, device=dev)
    lin.gated_norm([(x.view(n, -1).to(dev, dt), None, ga, z[:, :cut], dict(act="sigmoid", norm_cols=0, scale=0.7, spec=spec)),
                    (right.to(dev), w.to(dev, dt), gb, z[:, cut:], dict(act="sigmoid", norm_cols=cols, eps=eps, scale=1.3))])
    close(z[:, :heads * vdim], 0.7 * left.reshape(n, -1) * oracle.sigmoid(g1), dt)
    close(z[:, cut:cut + cols], 1.3 * oracle.rms(right, eps) * w * oracle.sigmoid(g2), dt)
    assert not z[:, heads * vdim:cut].any() and not z[:, cut + cols:].any()
    # a norm per head with shared gains and a SiLU gate
    hv = heads * vdim
    wh = rnd(vdim, seed=5, dtype=dt)
    z = torch.empty(n, hv, dtype=dt, device=dev)
    lin.gated_norm([(left.reshape(n, -1).to(dev), wh.to(dev, dt), ga, z, dict(act="silu", norm_cols=vdim, eps=eps, scale=1.0))])
    close(z, (oracle.rms(left, eps) * wh).reshape(n, -1) * oracle.silu(g1), dt)


# ------------------------------------------------------------------ attention with a distance bias

def attention_case(spec, kv_lens, qlens, page, dev, dt, seed=0, stand_out=True):
    """Normed rows in pages, with one far and one near key per sequence that a query matches strongly."""
    total, D = sum(-(-n // page) for n in kv_lens), spec.head_dim
    order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.zeros(total + 1, 2, spec.kv_heads, page, D)
    qs, ks, vs, tables = [], [], [], []
    for i, (n, ql) in enumerate(zip(kv_lens, qlens)):
        q = rnd(ql, spec.heads, spec.dim, seed=seed + 10 * i + 1, dtype=dt)
        k, v = rnd(n, spec.kv_heads, spec.dim, seed=seed + 10 * i + 2, dtype=dt), rnd(n, spec.kv_heads, spec.vdim, seed=seed + 10 * i + 3, dtype=dt)
        if stand_out:
            # every query finds the keys on both sides of its window's edge and at a page's border far more alike than the rest
            u = rnd(spec.dim, seed=99, dtype=dt)
            for t in range(ql):
                pos = n - ql + t
                q[t] += u
                for j in (pos, pos - spec.window + 1, pos - spec.window, pos // page * page):
                    if 0 <= j < n and (t in (0, ql // 2, ql - 1)):
                        k[j] = (2.0 * u).to(dt).float()
        q = q.to(dt).float()
        table = [order.pop() for _ in range(-(-n // page))]
        for j in range(n):
            cache[table[j // page], 0, :, j % page, :spec.dim] = k[j]
            cache[table[j // page], 1, :, j % page, :spec.vdim] = v[j]
        qs.append(q); ks.append(k); vs.append(v); tables.append(table)
    indptr = np.concatenate([[0], np.cumsum([len(t) for t in tables])]).astype(np.int32)
    batch = ops.AttnBatch(np.concatenate([[0], np.cumsum(qlens)]).astype(np.int32), indptr,
                          np.concatenate(tables).astype(np.int32), np.asarray(kv_lens, np.int32), None, spec.window - 1)
    rows = torch.zeros(sum(qlens), spec.kv_heads, spec.group_pad, D)
    rows[:, :, :spec.group, :spec.dim] = torch.cat(qs).view(-1, spec.kv_heads, spec.group, spec.dim)
    return qs, ks, vs, batch, rows.view(sum(qlens), -1, D).to(dev, dt), cache.to(dev, dt)


def plain_attention(spec, rel, qs, ks, vs):
    out = []
    for q, k, v in zip(qs, ks, vs):
        n, ql = k.shape[0], q.shape[0]
        kk, vv = k.repeat_interleave(spec.group, 1), v.repeat_interleave(spec.group, 1)
        s = oracle.softcap(torch.einsum("ihd,jhd->hij", q, kk) * spec.scale, spec.softcap)
        s = s + oracle.distance_bias(n, rel, spec.bias_max)[:, n - ql:]
        full = torch.zeros(spec.heads, n, n)
        full[:, n - ql:] = s
        p = oracle.windowed_softmax(full, spec.window)[:, n - ql:]
        out.append(torch.einsum("hij,jhd->ihd", p, vv))
    return torch.cat(out)


def spread(out, spec):
    n = out.shape[0]
    assert not out.view(n, spec.kv_heads, spec.group_pad, -1)[..., spec.vdim:].any()
    return out.view(n, spec.kv_heads, spec.group_pad, -1)[:, :, :spec.group, :spec.vdim].reshape(n, spec.heads, spec.vdim)


ATT = {"g3": (6, 2, 40, 24, 37, 90, 8.0, 12), "g1": (3, 3, 64, 64, 64, 130, 50.0, 32), "g4": (8, 2, 128, 128, 129, 300, 30.0, 16),
       "g8": (8, 1, 72, 100, 70, 150, 4.0, 8), "d256": (4, 2, 136, 200, 50, 90, 8.0, 10), "any": (20, 1, 24, 24, 60, 99, 8.0, 10),
       "huge": (2, 1, 264, 300, 33, 80, 8.0, 6), "one": (2, 2, 8, 16, 1, 9, 8.0, 4), "wide": (16, 1, 128, 96, 2000, 5000, 20.0, 32)}


def att_spec(name):
    h, kv, d, e, w, far, cap, rows = ATT[name]
    return BiasedAttentionSpec(h, kv, d, e, w, 1.3 * d ** -0.5, cap, far, rows)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("page", [16, 32])
def test_biased_attention_of_portions(path, name, page):
    """Prompts and portions of prompts: around the window's edge, over page and block borders, at the first tokens."""
    dev, dt = path
    spec = att_spec(name)
    if name == "wide" and dev == "cpu":
        pytest.skip("long")
    kv_lens, qlens = ([47, 1, 30, 64], [47, 1, 2, 20]) if dev == "cpu" else ([230, 1, 130, 64, 190], [230, 1, 2, 20, 100])
    if name == "wide":
        kv_lens, qlens = [2300], [300]
    rel = rnd(spec.buckets, spec.heads, seed=5, dtype=dt, std=1.5)
    qs, ks, vs, batch, q, cache = attention_case(spec, kv_lens, qlens, page, dev, dt)
    table, rs = lin.bias_table(rel, spec, dev), recurrent(batch.qo_indptr.tolist(), list(range(len(qlens))), [0] * len(qlens), dev)
    slots = torch.zeros(q.shape[0], dtype=torch.int32, device=dev)
    plan = batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, page, dev)
        plan.host = batch
    got = lin.biased_attention(q, cache, table, plan, rs, slots, spec)
    close(spread(got, spec), plain_attention(spec, rel, qs, ks, vs), dt, bf16=1e-2)
    if dev != "cpu":
        ops.check_kernel_status()


@pytest.mark.parametrize("path", PATHS[1:])
@pytest.mark.parametrize("name", list(ATT))
def test_biased_attention_of_decode_steps(path, name):
    """Contexts of many lengths in one decode step: their keys split over work items; a window wider than the layer's in the plan."""
    dev, dt = path
    spec = att_spec(name)
    w = spec.window
    kv_lens = sorted({1, 2, 15, 16, 17, max(1, w - 1), w, w + 1, w + 15, w + 16, 200, 333})
    rel = rnd(spec.buckets, spec.heads, seed=5, dtype=dt, std=1.5)
    qs, ks, vs, batch, q, cache = attention_case(spec, kv_lens, [1] * len(kv_lens), 16, dev, dt)
    r, sms = len(kv_lens), ops.num_sms()
    ir, st, en, indptr = ops.plan_decode_items(np.asarray(kv_lens), spec.kv_heads, 2 * sms, r + 16 * sms, window_left=w + 40)
    t = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    scratch = torch.empty(ops.decode_scratch_floats(r + 16 * sms, q.shape[1], spec.head_dim), device=dev)
    plan = ops.DecodePlan(t(batch.page_indices), t(batch.kv_page_indptr), t(ir), t(st), t(en), t(indptr), t([len(ir)]), scratch,
                          r + 16 * sms, r, 2 * sms, 16, w + 40, kv_lens=t(kv_lens))
    rs = recurrent(list(range(r + 1)), list(range(r)), [0] * r, dev)
    got = lin.biased_attention(q, cache, lin.bias_table(rel, spec, dev), plan, rs, torch.zeros(r, dtype=torch.int32, device=dev), spec)
    close(spread(got, spec), plain_attention(spec, rel, qs, ks, vs), dt, bf16=1e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "d256"])
def test_biased_attention_under_a_custom_mask(path, name):
    """A mask chooses among the keys of the window; later keys that it shows take the bias of distance 0."""
    dev, dt = path
    spec = att_spec(name)
    n, ql = 61, 30
    rel = rnd(spec.buckets, spec.heads, seed=5, dtype=dt)
    qs, ks, vs, batch, q, cache = attention_case(spec, [n], [ql], 16, dev, dt, stand_out=False)
    mask = torch.rand(ql, n, generator=torch.Generator().manual_seed(3)) < 0.4
    mask[:, n - ql:] |= torch.eye(ql, dtype=torch.bool)
    batch.masks = [mask.numpy()]
    table, rs = lin.bias_table(rel, spec, dev), recurrent([0, ql], [0], [0], dev)
    plan = batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, 16, dev)
        plan.host = batch
        plan.mask_bits, plan.mask_word_indptr = ops.pack_masks([mask.numpy()], [n], dev)
    got = spread(lin.biased_attention(q, cache, table, plan, rs, torch.zeros(ql, dtype=torch.int32, device=dev), spec), spec)
    kk, vv = ks[0].repeat_interleave(spec.group, 1), vs[0].repeat_interleave(spec.group, 1)
    gap = torch.arange(n - ql, n)[:, None] - torch.arange(n)[None]
    rows = torch.tensor([oracle.distance_bucket(max(0, i), spec.buckets, spec.bias_max) for i in range(n)])
    s = oracle.softcap(torch.einsum("ihd,jhd->hij", qs[0], kk) * spec.scale, spec.softcap) + rel[rows][gap.clamp(min=0)].permute(2, 0, 1)
    p = torch.softmax(s.masked_fill(~mask[None] | (gap >= spec.window)[None], float("-inf")), -1)
    close(got, torch.einsum("hij,jhd->ihd", p, vv), dt, bf16=1e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "g8", "d256", "one"])
def test_rows_normed_over_the_whole_projection(path, name):
    dev, dt = path
    spec, n, page, eps = att_spec(name), 9, 16, 1e-3
    nq, nk, nv = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim
    q, k, v = rnd(n, nq, dtype=dt, std=3), rnd(n, nk, seed=1, dtype=dt, std=0.1), rnd(n, nv, seed=2, dtype=dt)
    wq, wk = rnd(nq, seed=3, dtype=dt), rnd(nk, seed=4, dtype=dt)
    slots = torch.tensor([4, 9, 0, 31, 17, 2, -1, 30, 16], dtype=torch.int32)
    cache = torch.full((3, 2, spec.kv_heads, page, spec.head_dim), 7.0, dtype=dt, device=dev)
    if dev == "cpu":
        cache.zero_()
    got = lin.biased_rows(*padded([q, k, v], dev, dt), wq.to(dev, dt), wk.to(dev, dt), slots.to(dev), cache, spec, eps)
    rows = got.view(n, spec.kv_heads, spec.group_pad, spec.head_dim).float().cpu()
    close(rows[:, :, :spec.group, :spec.dim].reshape(n, nq), oracle.rms(q, eps) * wq, dt)
    assert not rows[:, :, spec.group:].any() and not rows[..., spec.dim:].any()
    kn = (oracle.rms(k, eps) * wk).view(n, spec.kv_heads, spec.dim)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            at = cache[s // page, :, :, s % page].float().cpu()
            close(at[0, :, :spec.dim], kn[i], dt)
            close(at[1, :, :spec.vdim], v[i].view(spec.kv_heads, spec.vdim), dt)
            assert not at[0, :, spec.dim:].any() and not at[1, :, spec.vdim:].any()


# ------------------------------------------------------------------ experts, stream
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("experts,identity,top,ff,width,n", [(5, 3, 3, 40, 96, 50), (1, 1, 2, 16, 48, 7), (4, 0, 1, 21, 100, 300),
                                                             (40, 9, 6, 32, 64, 33), (3, 60, 5, 48, 320, 130)])
def test_experts_with_identity_outputs(path, experts, identity, top, ff, width, n):
    dev, dt = path
    s = ExpertsSpec(experts, identity, top, ff, 1.2)
    e, wp, fp = s.outputs, -(-width // 8) * 8, -(-ff // 16) * 16
    # choice scores on distinct levels, so that no rounding turns a choice
    h, router = rnd(n, width, dtype=dt), rnd(e, width, seed=1, dtype=dt, std=2 * width ** -0.5)
    corr = torch.randperm(e, generator=torch.Generator().manual_seed(2)).float() * 0.3
    w = {"router": router, "correction": corr}
    for i in range(experts):
        for j, name in ((10, "gate"), (90, "up")):
            w[f"e{i}.{name}"] = rnd(ff, width, seed=j + i, dtype=dt, std=1.5 * width ** -0.5)
        w[f"e{i}.down"] = rnd(width, ff, seed=170 + i, dtype=dt, std=ff ** -0.5)
    ref = oracle.moe(h, w, {"router": {"experts": experts, "top": top}, "expert": {"limit": 1.2}})
    gu, down = torch.zeros(experts, 2 * fp, wp), torch.zeros(experts, wp, fp)
    for i in range(experts):
        gu[i, 0:2 * ff:2, :width], gu[i, 1:2 * ff:2, :width], down[i, :width, :ff] = w[f"e{i}.gate"], w[f"e{i}.up"], w[f"e{i}.down"]
    x = torch.nn.functional.pad(h, (0, wp - width)).to(dev, dt)
    rp = torch.nn.functional.pad(router, (0, wp - width)).to(dev, dt)
    gu, down, c = gu.to(dev, dt), down.to(dev, dt), corr.to(dev)
    if dt == BF16:
        buf = ops.MoeBuffers(512, wp, fp, experts, top, dev)
        for _ in range(2):          # the second pass finds the counters as the first left them
            got = lin.scored_experts(x, rp, c, gu, down, s, buf)
    else:
        got = lref.experts(x, x @ rp.t(), c, gu, down, s)
    close(got[:, :width], ref, dt, bf16=1.5e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("width", [64, 100, 102, 2560])
def test_output_norm_layer_scale_and_next_norm_in_one_pass(path, width):
    """x += norm(y) * (1 + w) * ls; h = norm(x) * (1 + w'), gains in 32-bit."""
    dev, dt = path
    n, ld, eps = 11, -(-width // 8) * 8, 1e-4
    x, y = rnd(n, width), rnd(n, width, seed=1, dtype=dt, std=5)
    wb, ls, w2 = rnd(width, seed=2, dtype=dt, std=0.3), rnd(width, seed=3, dtype=dt), rnd(width, seed=4, dtype=dt, std=0.3)
    xs = x + oracle.norm_about_one(y, wb, eps) * ls
    pad = lambda t, d: torch.nn.functional.pad(t, (0, ld - width)).to(dev, d)
    gx, gh, _ = lops.stream_norm(pad(x, F32), width, eps, pad(y, dt), ((1 + wb) * ls).to(dev), (1 + w2).to(dev), dtype=dt)
    close(gx[:, :width], xs, F32)
    close(gh[:, :width], oracle.norm_about_one(xs, w2, eps), dt, bf16=4e-3)
    assert gh.dtype == dt and not gh[:, width:].any()


@pytest.mark.parametrize("path", PATHS)
def test_embedding_scale(path):
    dev, dt = path
    table = rnd(13, 20, dtype=dt)
    x = lops.stream_embed(torch.tensor([12, 0, 5], dtype=torch.int32, device=dev), table.to(dev, dt), 24, 13.5)
    assert torch.equal(x[:, :20].cpu(), table[[12, 0, 5]] * 13.5) and not x[:, 20:].any()


@gpu
def test_long_constant_decay_does_not_drift():
    """A head that forgets nothing and one that forgets slowly over thousands of tokens, prompt against steps."""
    n, h, d, e = 4096, 2, 16, 32
    decay = torch.tensor([1.0, 0.9995])
    q, k, v = rnd(n, h * d, dtype=BF16), rnd(n, h * d, seed=1, dtype=BF16, std=0.1), rnd(n, h * e, seed=2, dtype=BF16)
    spec = LightningSpec(h, d, e, decay.tolist())
    a = decay.double()[None, :, None].expand(n, h, d)
    states = []
    ref = oracle.decayed_state(*(x.double().view(n, h, -1) for x in (q, k, v)), a, states).reshape(n, -1)
    for dt in (BF16, F32):
        state = torch.zeros(1, spec.state_elems, device="cuda")
        qq, kk, vv = padded([q, k, v], "cuda", dt)
        got = lin.linear_attention(qq, kk, vv, spec, recurrent([0, n], [0], [1], "cuda"), state, False, head_decay=decay.cuda())
        close(got, ref, dt, f32=1e-5, bf16=2e-3)
        close(state[0].view(h, d, e), states[-1], dt, f32=1e-5, bf16=2e-3)
