"""Each mechanism of the Nukelix blocks alone: the ops of pie_b200.ops.{grouped,linear,latent} against the plain functions
in nukelix_oracle.py, on the CPU path and on the kernels."""
import numpy as np
import nukelix_oracle as oracle
import pytest
import torch

from pie_b200 import ops
from pie_b200.driver.recurrent import RecurrentInputs
from pie_b200.models.block_spec import EVERYTHING, ExpertsSpec, GroupedAttentionSpec, LatentSpec, MatrixMemorySpec, RotarySpec
from pie_b200.models.nukelix import _WAVELENGTH, _YARN, _scaling
from pie_b200.ops import grouped, latent as lops, linear as lin, linear_reference as lref

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


# ------------------------------------------------------------------ rotation
@pytest.mark.parametrize("dims,base,s", [(24, 300.0, (6.0, 1.0, 3.0, 48)), (64, 1e4, (8.0, 1.0, 4.0, 8192)), (2, 9.0, (2.0, 1.0, 2.0, 5)),
                                         (16, 50.0, (4.0, 2.0, 2.5, 300))])
def test_frequencies_stretched_by_wavelength(dims, base, s):
    d = dict(zip(("factor", "low", "high", "original"), s))
    r = RotarySpec(dims, base, True, _scaling({"scaling": d}, "llama3", _WAVELENGTH))
    want = oracle.stretched_by_wavelength(oracle.frequencies({"dims": dims, "base": base}), **d)
    assert torch.equal(r.frequencies(), want.float()) and r.factor == 1.0


@pytest.mark.parametrize("dims,base,s", [(32, 700.0, (4.0, 64, 8.0, 1.0)), (64, 1e4, (40.0, 4096, 32.0, 1.0)), (2, 9.0, (2.0, 30, 3.0, 1.0)),
                                         (20, 1e6, (1.0, 100, 2.0, 1.5)), (8, 30.0, (3.0, 7, 32.0, 20.0))])
def test_frequencies_stretched_by_index(dims, base, s):
    d = dict(zip(("factor", "original", "fast", "slow"), s))
    r = RotarySpec(dims, base, True, _scaling({"scaling": d}, "yarn", _YARN))
    want, factor = oracle.stretched_by_index(oracle.frequencies({"dims": dims, "base": base}), {"dims": dims, "base": base}, **d)
    assert torch.allclose(r.frequencies(), want.float(), rtol=1e-6, atol=0) and r.factor == pytest.approx(factor)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("dim,rot,dims,heads,rank", [(24, 12, 12, 3, 40), (33, 6, 4, 2, 50), (16, 16, 16, 1, 16)])
def test_latent_rows_with_neighbouring_pairs(path, dim, rot, dims, heads, rank):
    """Queries and latent rows of separate projections; cos and sin carry a factor."""
    dev, dt = path
    rot_d = {"dims": dims, "base": 60.0, "scaling": {"factor": 4.0, "original": 40, "fast": 6.0, "slow": 1.0}}
    s = LatentSpec(heads, dim, rot, 16, rank, EVERYTHING, 0.3, 60.0, dims, q_rank=8, rot_adjacent=True,
                   rot_scaling=_scaling(rot_d, "yarn", _YARN))
    n = 8
    q, kv, nw = rnd(n, s.q_rows, dtype=dt, std=2), rnd(n, rank + rot, seed=1, dtype=dt, std=2), rnd(rank, seed=2, dtype=dt)
    pos = [0, 1, 2, 5, 63, 64, 1000, 4095]
    slots = torch.tensor([4, 9, 0, 31, -1, 2, 17, 30], dtype=torch.int32)
    cache = torch.full((2, 16, s.row), 7.0, dtype=dt, device=dev)
    qq, kk = padded([q, kv], dev, dt)
    got = lops.latent_rows(qq, torch.tensor(pos, dtype=torch.int32, device=dev), slots.to(dev), s.rotary.frequencies(dev), nw.to(dev, dt),
                           cache, s, 1e-5, s.row, s.rank_pad, False, kk)
    f, factor = oracle.stretched_by_index(oracle.frequencies(rot_d), rot_d, **rot_d["scaling"])
    turn = lambda x: oracle.rotated(x, f, True, factor, pos)
    close(got[..., s.rank_pad:s.rank_pad + rot], turn(q.view(n, heads, dim + rot)[..., dim:]), dt, f32=3e-4)
    c, kr, flat = oracle.gained_norm(kv[:, :rank], nw, 1e-5), turn(kv[:, rank:]), cache.view(32, -1)
    for i, at in enumerate(slots.tolist()):
        if at >= 0:
            close(flat[at, :rank], c[i], dt)
            close(flat[at, s.rank_pad:s.rank_pad + rot], kr[i], dt, f32=3e-4)


# ------------------------------------------------------------------ grouped attention
ATT = {"g3": (6, 2, 40, 24, 24, 37, 5, True), "g1": (3, 3, 64, 64, 64, 64, 64, True), "g4": (8, 2, 128, 128, 64, 129, 70, True),
       "g8": (8, 1, 72, 100, 20, 70, 1, False), "d256": (4, 2, 136, 200, 136, 50, 17, True), "any": (20, 1, 24, 24, 8, 60, 9, True),
       "huge": (2, 1, 264, 300, 2, 33, 2, True), "one": (2, 2, 8, 16, 8, 1, 1, True), "nothing kept": (16, 1, 128, 96, 128, 100, 0, True),
       "everything": (6, 3, 64, 48, 64, EVERYTHING, 0, False), "all and a sink": (4, 1, 96, 32, 24, EVERYTHING, 0, True)}


def att_spec(name, adjacent=True):
    h, kv, d, e, rot, w, keep, sink = ATT[name]
    return GroupedAttentionSpec(h, kv, d, e, 1.2 * d ** -0.5, RotarySpec(rot, 200.0, adjacent), w, keep, sink)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "g8", "d256", "one", "huge"])
@pytest.mark.parametrize("adjacent", [True, False])
@pytest.mark.parametrize("mix", ["source", "mixed", "none"])
def test_rows_biased_normed_rotated_and_mixed(path, name, adjacent, mix):
    dev, dt = path
    spec, n, page, eps = att_spec(name, adjacent), 9, 16, 1e-3
    nq, nk, nv = spec.heads * spec.dim, spec.kv_heads * spec.dim, spec.kv_heads * spec.vdim
    h = {"heads": spec.heads, "kv_heads": spec.kv_heads}
    parts = {"q": rnd(n, nq, dtype=dt, std=3), "k": rnd(n, nk, seed=1, dtype=dt, std=0.1), "v": rnd(n, nv, seed=2, dtype=dt)}
    w = {"q.b": rnd(nq, seed=3, dtype=dt), "k.b": rnd(nk, seed=4, dtype=dt, std=0.1), "v.b": rnd(nv, seed=5, dtype=dt),
         "q.norm": rnd(nq, seed=6, dtype=dt), "k.norm": rnd(nk, seed=7, dtype=dt)}
    for k, x in parts.items():              # the projections' products themselves: their weights are unit matrices
        w[k] = torch.eye(x.shape[1])
    pos = [0, 1, 2, 5, 63, 64, 1000, 4095, 7]
    slots = torch.tensor([4, 9, 0, 31, 17, 2, -1, 30, 16], dtype=torch.int32)
    cache = torch.full((3, 2, spec.kv_heads, page, spec.head_dim), 0.0 if dev == "cpu" else 7.0, dtype=dt, device=dev)
    lw = {k.replace(".", "_"): v.to(dev, dt) for k, v in w.items()}
    lw["rope"] = spec.rot.frequencies(dev)
    first = rnd(n, nv, seed=8)
    got, kept = grouped.grouped_rows(*padded(list(parts.values()), dev, dt), lw, torch.tensor(pos, dtype=torch.int32, device=dev), slots.to(dev),
                                     cache, spec, eps, first.to(dev) if mix == "mixed" else None, 0.3, mix == "source")
    f = oracle.frequencies({"dims": spec.rot.dims, "base": 200.0})
    q, k, v = (oracle.projected_heads(parts[x], w, h, eps, x) for x in "qkv")
    q, k = oracle.rotated(q, f, adjacent, 1.0, pos), oracle.rotated(k, f, adjacent, 1.0, pos)
    rows = got.view(n, spec.kv_heads, spec.group_pad, spec.head_dim).float().cpu()
    close(rows[:, :, :spec.group, :spec.dim].reshape(n, spec.heads, spec.dim), q, dt, f32=3e-4)
    assert not rows[:, :, spec.group:].any() and not rows[..., spec.dim:].any()
    if mix == "source":
        close(kept, v.reshape(n, -1), F32)
    if mix == "mixed":
        v = oracle.mixed_values(v, first.view(v.shape), 0.3)
    for i, s in enumerate(slots.tolist()):
        if s >= 0:
            at = cache[s // page, :, :, s % page].float().cpu()
            close(at[0, :, :spec.dim], k[i], dt, f32=3e-4)
            close(at[1, :, :spec.vdim], v[i], dt)
            assert not at[0, :, spec.dim:].any() and not at[1, :, spec.vdim:].any()


def attention_case(spec, kv_lens, qlens, page, dev, dt, seed=0):
    """Rows in shuffled pages, with keys that a query finds far more alike than the rest: on both sides of the edge of its
    window and of the kept tokens, and at a page's border."""
    total, D = sum(-(-n // page) for n in kv_lens), spec.head_dim
    order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.zeros(total + 1, 2, spec.kv_heads, page, D)
    qs, ks, vs, tables = [], [], [], []
    u = rnd(spec.dim, seed=99, dtype=dt)
    for i, (n, ql) in enumerate(zip(kv_lens, qlens)):
        q = rnd(ql, spec.heads, spec.dim, seed=seed + 10 * i + 1, dtype=dt)
        k, v = rnd(n, spec.kv_heads, spec.dim, seed=seed + 10 * i + 2, dtype=dt), rnd(n, spec.kv_heads, spec.vdim, seed=seed + 10 * i + 3, dtype=dt)
        for t in (0, ql // 2, ql - 1):
            pos = n - ql + t
            q[t] += 0.6 * u
            for j in (pos, pos - spec.window + 1, pos - spec.window, pos // page * page, spec.keep_first - 1, spec.keep_first):
                if 0 <= j < n:
                    k[j] = (1.5 * u).to(dt).float()
        q = q.to(dt).float()
        table = [order.pop() for _ in range(-(-n // page))]
        for j in range(n):
            cache[table[j // page], 0, :, j % page, :spec.dim] = k[j]
            cache[table[j // page], 1, :, j % page, :spec.vdim] = v[j]
        qs.append(q), ks.append(k), vs.append(v), tables.append(table)
    indptr = np.concatenate([[0], np.cumsum([len(t) for t in tables])]).astype(np.int32)
    batch = ops.AttnBatch(np.concatenate([[0], np.cumsum(qlens)]).astype(np.int32), indptr, np.concatenate(tables).astype(np.int32),
                          np.asarray(kv_lens, np.int32), None, -1)
    rows = torch.zeros(sum(qlens), spec.kv_heads, spec.group_pad, D)
    rows[:, :, :spec.group, :spec.dim] = torch.cat(qs).view(-1, spec.kv_heads, spec.group, spec.dim)
    return qs, ks, vs, batch, rows.view(sum(qlens), -1, D).to(dev, dt), cache.to(dev, dt)


def plain_attention(spec, qs, ks, vs):
    out = []
    for q, k, v in zip(qs, ks, vs):
        n, ql = k.shape[0], q.shape[0]
        kk, vv = k.repeat_interleave(spec.group, 1), v.repeat_interleave(spec.group, 1)
        full = torch.zeros(spec.heads, n, n)
        full[:, n - ql:] = torch.einsum("ihd,jhd->hij", q, kk) * spec.scale
        see = oracle.visible(n) if spec.window == EVERYTHING else oracle.visible(n, spec.window, spec.keep_first)
        out.append(torch.einsum("hij,jhd->ihd", oracle.weights_over_keys(full, see, spec.sink)[:, n - ql:], vv))
    return torch.cat(out)


def spread(out, spec):
    n = out.shape[0]
    assert not out.view(n, spec.kv_heads, spec.group_pad, -1)[..., spec.vdim:].any()
    return out.view(n, spec.kv_heads, spec.group_pad, -1)[:, :, :spec.group, :spec.vdim].reshape(n, spec.heads, spec.vdim)


def sinks(spec, dev):
    return torch.zeros(spec.kv_heads * spec.group_pad, device=dev) if spec.sink else None


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("page", [16, 32])
def test_grouped_attention_of_portions(path, name, page):
    """Prompts and portions of prompts: around the edges of the window and of the kept tokens, over page and block borders."""
    dev, dt = path
    spec = att_spec(name)
    kv_lens, qlens = ([47, 1, 30, 64, 90], [47, 1, 2, 20, 3]) if dev == "cpu" else ([230, 1, 130, 64, 390, 700], [230, 1, 2, 20, 100, 5])
    qs, ks, vs, batch, q, cache = attention_case(spec, kv_lens, qlens, page, dev, dt)
    rs = recurrent(batch.qo_indptr.tolist(), list(range(len(qlens))), [0] * len(qlens), dev)
    plan = batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, page, dev)
        plan.host = batch
    got = grouped.grouped_attention(q, cache, plan, rs, torch.zeros(q.shape[0], dtype=torch.int32, device=dev), spec, sinks(spec, dev))
    close(spread(got, spec), plain_attention(spec, qs, ks, vs), dt, bf16=1.2e-2)
    if dev != "cpu":
        ops.check_kernel_status()


@pytest.mark.parametrize("path", PATHS[1:])
@pytest.mark.parametrize("name", list(ATT))
@pytest.mark.parametrize("even", [True, False])
def test_grouped_attention_of_decode_steps(path, name, even):
    """Contexts of many lengths in one decode step, their keys split over work items that the layer's window hides in part."""
    dev, dt = path
    spec = att_spec(name)
    w, keep = min(spec.window, 150), spec.keep_first
    kv_lens = sorted({1, 2, 15, 16, 17, max(1, w - 1), w, w + 1, w + 15, w + 16, w + keep, w + keep + 1, w + keep + 17, 200, 333, 900})
    qs, ks, vs, batch, q, cache = attention_case(spec, kv_lens, [1] * len(kv_lens), 16, dev, dt)
    r, sms = len(kv_lens), ops.num_sms()
    if even:
        ir, st, en, indptr, _ = ops.plan_even_items(np.asarray(kv_lens), sms, r + 16 * sms, min_keys=32)
    else:
        ir, st, en, indptr = ops.plan_decode_items(np.asarray(kv_lens), spec.kv_heads, 2 * sms, r + 16 * sms)
    t = lambda a: torch.as_tensor(np.asarray(a, np.int32)).to(dev)
    scratch = torch.full((ops.decode_scratch_floats(r + 16 * sms, q.shape[1], spec.head_dim),), float("nan"), device=dev)
    plan = ops.DecodePlan(t(batch.page_indices), t(batch.kv_page_indptr), t(ir), t(st), t(en), t(indptr), t([len(ir)]), scratch,
                          r + 16 * sms, r, 2 * sms, 16, -1, kv_lens=t(kv_lens))
    rs = recurrent(list(range(r + 1)), list(range(r)), [0] * r, dev)
    got = grouped.grouped_attention(q, cache, plan, rs, torch.zeros(r, dtype=torch.int32, device=dev), spec, sinks(spec, dev))
    close(spread(got, spec), plain_attention(spec, qs, ks, vs), dt, bf16=1.2e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["g3", "d256"])
def test_grouped_attention_under_a_custom_mask(path, name):
    """A mask chooses among the keys of the window and the kept tokens."""
    dev, dt = path
    spec, n, ql = att_spec(name), 75, 30
    qs, ks, vs, batch, q, cache = attention_case(spec, [n], [ql], 16, dev, dt)
    mask = torch.rand(ql, n, generator=torch.Generator().manual_seed(3)) < 0.4
    mask[:, n - ql:] |= torch.eye(ql, dtype=torch.bool)
    batch.masks, plan = [mask.numpy()], batch
    if dev != "cpu":
        plan = ops.build_prefill_plan(batch, 1, 16, dev)
        plan.host = batch
        plan.mask_bits, plan.mask_word_indptr = ops.pack_masks([mask.numpy()], [n], dev)
    got = grouped.grouped_attention(q, cache, plan, recurrent([0, ql], [0], [0], dev), torch.zeros(ql, dtype=torch.int32, device=dev), spec,
                                    sinks(spec, dev))
    kk, vv = ks[0].repeat_interleave(spec.group, 1), vs[0].repeat_interleave(spec.group, 1)
    i, j = torch.arange(n - ql, n)[:, None], torch.arange(n)[None]
    see = mask & ((i - j < spec.window) | (j < spec.keep_first))
    p = oracle.weights_over_keys(torch.einsum("ihd,jhd->hij", qs[0], kk) * spec.scale, see, spec.sink)
    close(spread(got, spec), torch.einsum("hij,jhd->ihd", p, vv), dt, bf16=1.2e-2)


# ------------------------------------------------------------------ matrix memory
SHAPES = [(1, 1, 1), (3, 7, 11), (2, 32, 64), (2, 40, 24), (1, 128, 128), (3, 96, 36), (1, 200, 64), (1, 272, 24), (1, 64, 260)]


def memory_case(n, h, d, e, dt, kind, width=24):
    x, w = rnd(n, width, dtype=dt), rnd(2 * h, width, seed=1, dtype=dt, std=width ** -0.5)
    b = torch.cat([rnd(h, seed=2), 4.0 + rnd(h, seed=3)])
    if kind == "spikes":                        # now and then an input gate far above the others
        x[::29, 0], w[:h, 0] = 3.0, 4.0
    if kind == "forgetful":
        b[h:] -= 9.0
    return x, w, b, rnd(n, h * d, seed=4, dtype=dt), rnd(n, h * d, seed=5, dtype=dt, std=d ** -0.5), rnd(n, h * e, seed=6, dtype=dt)


def memory_oracle(x, w, b, q, k, v, h, cap, state=None):
    n = x.shape[0]
    i, f = oracle.log_gates(x.double(), {"i": w[:h].double(), "f": w[h:].double(), "i.b": b[:h].double(), "f.b": b[h:].double()}, cap)
    heads = lambda y: y.double().view(n, h, -1)
    return oracle.matrix_memory(heads(q) * (q.shape[1] // h) ** -0.5, heads(k), heads(v), i, f, state)


def run_memory(x, w, b, q, k, v, spec, rs, state, dev, dt, single):
    """o [N, H, V] as the mixer has it ahead of its norm."""
    decay, key, floor = lin.memory_gates(x.to(dev, dt), w.to(dev, dt), b.to(dev), spec, rs, state, single)
    qq, kk, vv = padded([q, k, v], dev, dt)
    o, den = lin.linear_attention(qq, kk, vv, spec, rs, state, single, q_scale=spec.dim ** -0.5, gates=(decay, key))
    return (o.view(len(x), spec.heads, spec.vdim) / (torch.maximum(den.abs(), floor) + 1e-6).t()[..., None]).cpu()


def same_heads(got, want, dt, bf16=1e-2):
    """Outputs whose denominators differ in size by token and head: each against its own root mean square."""
    want = want.float()
    rms = want.pow(2).mean(-1, keepdim=True).sqrt()
    e = ((got - want).abs() / (rms + 1e-3 * rms.max())).flatten(1).amax(1)
    limit = 3e-4 if dt == F32 else bf16
    # a numerator next to zero (q.k of the only key, say) magnifies a rounding: one token in twenty may
    assert (e > 10 * limit).sum() <= len(e) // 20 and e.median() <= limit, (float(e.median()), float(e.max()))


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("h,d,e", SHAPES)
@pytest.mark.parametrize("kind", ["steady", "spikes", "forgetful"])
def test_matrix_memory_in_portions(path, h, d, e, kind):
    """One sequence in portions of many sizes, whose state (matrix, normaliser, maximum) lives in one slot."""
    dev, dt = path
    sizes = [1, 2, 1, 3, 10, 23] if dev == "cpu" else [2, 64, 1, 1, 63, 65, 3, 17, 300, 84]
    x, w, b, q, k, v = memory_case(sum(sizes), h, d, e, dt, kind)
    spec = MatrixMemorySpec(h, d, e, 6.0)
    ref, (s, nrm, m) = memory_oracle(x, w, b, q, k, v, h, 6.0)
    cache = torch.full((3, -(-spec.state_elems // 4) * 4 + 8), float("nan"), device=dev)      # an unset slot must not leak in
    state, at, out = cache[:, 4:4 + spec.state_elems], 0, []
    for size in sizes:
        rs = recurrent([0, size], [1], [1 if at == 0 else 0], dev)
        part = slice(at, at + size)
        out.append(run_memory(x[part], w, b, q[part], k[part], v[part], spec, rs, state, dev, dt, size == 1))
        at += size
    same_heads(torch.cat(out), ref, dt)
    got = state[1].cpu()
    close(got[-h:], m, F32, f32=1e-5 if dt == F32 else 2e-3)
    close(got[:h * d * e].view(h, d, e), s, dt)
    close(got[h * d * e:h * d * (e + 1)].view(h, d), nrm, dt)
    assert not state[0].isfinite().any() and not state[2].isfinite().any()


@pytest.mark.parametrize("path", PATHS)
def test_matrix_memory_over_a_ragged_batch(path):
    """Unequal portions in one launch: fresh and continued slots, a padding row, states of their own."""
    dev, dt = path
    h, d, e = 2, 24, 40
    spec = MatrixMemorySpec(h, d, e, 9.0)
    lens = [5, 1, 0, 33, 2] if dev == "cpu" else [70, 1, 0, 600, 2]
    slots, reset = [3, -1, 0, 4, 1], [1, 0, 0, 0, 1]
    qo = np.concatenate([[0], np.cumsum(lens)]).tolist()
    x, w, b, q, k, v = memory_case(qo[-1], h, d, e, dt, "spikes")
    before = rnd(6, spec.state_elems, seed=9)
    state = before.clone().to(dev)
    got = run_memory(x, w, b, q, k, v, spec, recurrent(qo, slots, reset, dev), state, dev, dt, False)
    for r, (a, z) in enumerate(zip(qo, qo[1:])):
        if slots[r] < 0 or a == z:
            continue
        old = before[slots[r]].double()
        start = None if reset[r] else (old[:h * d * e].view(h, d, e), old[h * d * e:h * d * (e + 1)].view(h, d), old[-h:])
        want, (s, nrm, m) = memory_oracle(x[a:z], w, b, q[a:z], k[a:z], v[a:z], h, 9.0, start)
        if z - a > 20:
            same_heads(got[a:z], want, dt)
        end = state[slots[r]].cpu()
        close(end[-h:], m, F32, f32=1e-5 if dt == F32 else 2e-3)
        close(end[:h * d * e].view(h, d, e), s, dt)
        close(end[h * d * e:h * d * (e + 1)].view(h, d), nrm, dt)
    for s in (0, 2, 5):
        assert torch.equal(state[s].cpu(), before[s])


@pytest.mark.parametrize("path", PATHS)
def test_gates_of_single_tokens_and_portions(path):
    """The factors and the floor themselves, over a long portion and token by token; a padding row stays out."""
    dev, dt = path
    h, n, cap = 3, 70 if dev == "cpu" else 2500, 4.0
    spec = MatrixMemorySpec(h, 2, 2, cap)
    x, w, b, *_ = memory_case(n, h, 2, 2, dt, "spikes")
    i, f = oracle.log_gates(x.double(), {"i": w[:h].double(), "f": w[h:].double(), "i.b": b[:h].double(), "f.b": b[h:].double()}, cap)
    m, want = torch.zeros(h, dtype=torch.double), []
    for t in range(n):
        new = torch.maximum(f[t] + m, i[t])
        want.append(torch.stack([f[t] + m - new, i[t] - new, torch.exp(-new)]))
        m = new
    want = torch.stack(want, 1)
    xs, ws, bs = x.to(dev, dt), w.to(dev, dt), b.to(dev)
    state = torch.zeros(3, spec.state_elems, device=dev)
    whole = torch.stack(lin.memory_gates(xs, ws, bs, spec, recurrent([0, n], [2], [1], dev), state, False)).cpu()
    steps, short = [], 40
    for t in range(short):
        rs = recurrent([0, 1, 2], [1, -1], [1 if t == 0 else 0, 0], dev)
        steps.append(torch.stack(lin.memory_gates(xs[[t, t]], ws, bs, spec, rs, state, True))[..., 0].cpu())
    want = want.transpose(1, 2)
    for got, ref in ((whole, want), (torch.stack(steps, -1), want[..., :short])):
        close(got[0] * np.log(2), ref[0], F32, f32=2e-5)
        close(got[1] * np.log(2), ref[1], F32, f32=2e-5)
        close(got[2], ref[2], F32, f32=2e-5)
    close(state[2, -h:], m, F32)
    assert not state[0].any()


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("heads,kv,vdim,rh,rv", [(6, 2, 24, 3, 40), (5, 1, 33, 2, 11), (4, 4, 8, 1, 64), (2, 2, 1, 2, 4)])
def test_gates_per_head_and_norm_of_a_quotient(path, heads, kv, vdim, rh, rv):
    """Attention heads gated by one number each beside a memory's heads: normed quotient, gains, elementwise gate; and a norm
    without a gate."""
    dev, dt = path
    n, eps = 7, 1e-3
    spec = GroupedAttentionSpec(heads, kv, 8, vdim, 1.0, RotarySpec(2, 10.0))
    left, right = rnd(n, heads, vdim, dtype=dt), rnd(n, rh, rv, seed=1)
    den, floor = rnd(n, rh, seed=2, std=2), rnd(n, rh, seed=3).abs()
    den[0], floor[0] = 0.0, 1e-4
    g1, g2, w = rnd(n, heads, seed=4, dtype=dt, std=2), rnd(n, rh * rv, seed=5, dtype=dt, std=2), rnd(rh * rv, seed=6, dtype=dt)
    x = torch.full((n, kv, spec.group_pad, spec.head_dim), 9.0)
    x[:, :, :spec.group, :vdim] = left.view(n, kv, spec.group, vdim)
    ga, gb = padded([g1, g2], dev, dt)
    cut = -(-heads * vdim // 8) * 8
    z = torch.full((n, cut + rh * rv + 8), 5.0, dtype=dt, device=dev)
    lin.gated_norm([(x.view(n, -1).to(dev, dt), None, ga, z[:, :cut], dict(act="sigmoid", norm_cols=0, scale=0.7, spec=spec, gate_cols=vdim)),
                    (right.reshape(n, -1).to(dev), w.to(dev, dt), gb, z[:, cut:],
                     dict(act="sigmoid", norm_cols=rv, eps=eps, scale=1.3, den=den.t().contiguous().to(dev), floor=floor.t().contiguous().to(dev)))])
    close(z[:, :heads * vdim], 0.7 * oracle.head_gate(left, g1, torch.eye(heads)).reshape(n, -1), dt)
    o = right / (torch.maximum(den.abs(), floor) + 1e-6)[..., None]
    close(z[:, cut:cut + rh * rv], 1.3 * oracle.rms(o, eps).reshape(n, -1) * w * oracle.sigmoid(g2), dt)
    assert not z[:, heads * vdim:cut].any() and not z[:, cut + rh * rv:].any()
    (c,) = padded([g2], dev, dt)
    z = torch.full((n, rh * rv + 3), 5.0, dtype=dt, device=dev)
    lin.gated_norm([(c, w.to(dev, dt), None, z, dict(norm_cols=rh * rv, cols=rh * rv, eps=eps, scale=1.0))])
    close(z[:, :rh * rv], oracle.gained_norm(g2, w, eps), dt)
    assert not z[:, rh * rv:].any()


# ------------------------------------------------------------------ experts, stream, logits
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("experts,top,ff,width,n,shared", [(5, 3, 40, 96, 50, 56), (1, 1, 16, 48, 7, 8), (4, 1, 21, 100, 300, 0),
                                                           (40, 6, 32, 64, 33, 24), (3, 3, 48, 320, 130, 40)])
def test_experts_that_read_weighted_inputs(path, experts, top, ff, width, n, shared):
    dev, dt = path
    s = ExpertsSpec(experts, 0, top, ff, None, "sigmoid", True, shared)
    wp, fp, sp = -(-width // 8) * 8, -(-ff // 16) * 16, -(-shared // 16) * 16
    # scores half apart, so that no rounding turns a choice; some saturate
    order = torch.stack([torch.randperm(experts, generator=torch.Generator().manual_seed(i)) for i in range(n)]).float()
    h = rnd(n, width, dtype=dt)
    if experts <= width:
        h[:, :experts] = (0.5 * order - 0.4 * experts).to(dt).float()
    router = torch.eye(experts, width)
    w = {"router": router}
    for i, (e, k) in enumerate([(f"e{i}", ff) for i in range(experts)] + ([("shared", shared)] if shared else [])):
        for j, name, std in ((10, "gate", 2.0), (90, "up", 1.0)):
            w[f"{e}.{name}"] = rnd(k, width, seed=j + i, dtype=dt, std=std * width ** -0.5)
        w[e + ".down"] = rnd(width, k, seed=170 + i, dtype=dt, std=k ** -0.5)
    ref = oracle.experts(h, w, {"router": {"experts": experts, "top": top}, "shared": shared or None})

    def fused(e, k, kp):
        gu, down = torch.zeros(2 * kp, wp), torch.zeros(wp, kp)
        gu[0:2 * k:2, :width], gu[1:2 * k:2, :width], down[:width, :k] = w[e + ".gate"], w[e + ".up"], w[e + ".down"]
        return gu.to(dev, dt), down.to(dev, dt)
    pairs = [fused(f"e{i}", ff, fp) for i in range(experts)]
    gu, down = torch.stack([a for a, _ in pairs]), torch.stack([b for _, b in pairs])
    x = torch.nn.functional.pad(h, (0, wp - width)).to(dev, dt)
    rp = torch.nn.functional.pad(router, (0, wp - width)).to(dev, dt)
    extra = None
    if shared:
        a, b = fused("shared", shared, sp)
        y = x.float() @ a.float().t()
        extra = ((oracle.silu(y[:, 0::2]) * y[:, 1::2]).to(dt).float() @ b.float().t()).to(dt)
    if dt == BF16:
        buf = ops.MoeBuffers(512, wp, fp, experts, top, dev)
        for _ in range(2):          # the second pass finds the counters as the first left them
            got = lin.sigmoid_experts(x, rp, gu, down, s, buf, extra)
    else:
        got = lref.sigmoid_experts(x, x @ rp.t(), gu, down, s)
        got = got if extra is None else got + extra
    close(got[:, :width], ref, dt, bf16=1.5e-2)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("width", [64, 100, 102, 2560])
def test_output_norm_and_a_copy_of_the_stream(path, width):
    """x += norm(y) * w; h = x in the activation type; without y only the copy."""
    dev, dt = path
    n, ld, eps = 11, -(-width // 8) * 8, 1e-4
    x, y, w = rnd(n, width), rnd(n, width, seed=1, dtype=dt, std=5), rnd(width, seed=2)
    pad = lambda t, d: torch.nn.functional.pad(t, (0, ld - width)).to(dev, d)
    gx, gh, _ = lops.stream_norm(pad(x, F32), width, eps, pad(y, dt), w.to(dev), dtype=dt, copy=True)
    close(gx[:, :width], x + oracle.gained_norm(y, w, eps), F32)
    assert torch.equal(gh, gx.to(dt)) and not gh[:, width:].any()
    gx, gh, _ = lops.stream_norm(pad(x, F32), width, eps, dtype=dt, copy=True)
    assert torch.equal(gx[:, :width].cpu(), x) and torch.equal(gh, gx.to(dt))


@pytest.mark.parametrize("path", PATHS)
def test_softcap_in_place_on_a_column_range(path):
    dev, dt = path
    y = rnd(5, 77, dtype=dt, std=40)
    wide = torch.nn.functional.pad(y, (0, 3), value=9.0).to(dev, dt)
    close(ops.softcap_(wide[:, :77], 25.0), oracle.soft_limit(y, 25.0), dt, bf16=4e-3)
    assert (wide[:, 77:] == 9.0).all()
