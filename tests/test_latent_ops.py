"""Each mechanism of the Puzutar blocks alone: the ops of pie_b200.ops.latent against the plain functions in
puzutar_oracle.py, on the CPU path and on the kernels (32-bit and bf16)."""
import numpy as np
import pytest
import puzutar_oracle as oracle
import torch

from pie_b200 import ops
from pie_b200.driver.recurrent import RecurrentInputs
from pie_b200.models.config import LatentSpec
from pie_b200.ops import latent as lops

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


def recurrent(qo, slots, reset, state, dev):
    t = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)
    r = len(qo) - 1
    req = np.repeat(np.arange(r), np.diff(qo)).tolist()
    return RecurrentInputs(t(qo), t(req), t(slots), t(reset), list(qo), list(slots), list(reset), None, None, {0: 0},
                           shift_state=state, shift_stage=torch.empty(r, state.shape[-1], device=dev) if dev != "cpu" else None)


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("width,groups", [(64, 1), (96, 3), (100, 5), (102, 6), (2560, 4), (4099, 1), (8192, 8)])
def test_stream_norm_shift_and_pending_token_input(path, width, groups):
    dev, dt = path
    n, ld, eps = 23, -(-width // 8) * 8, 1e-3
    x, y, yn, w, mix = rnd(n, width), rnd(n, width, seed=1, dtype=dt, std=3), rnd(width, seed=2, dtype=dt), rnd(width, seed=3, dtype=dt), \
        rnd(width, seed=4, dtype=dt)
    xs = x + oracle.rms(y, eps) * yn
    h = oracle.grouped_norm(xs, w, groups, eps)
    hs = oracle.token_shift(h, mix)
    pad = lambda t, d: torch.nn.functional.pad(t, (0, ld - width)).to(dev, d)
    args = (yn.to(dev, dt), w.to(dev, dt), groups, mix.to(dev, dt))
    state = torch.full((1, 3, width), float("nan"), device=dev)       # an unset slot must not leak in
    a = 0
    for size in (1, 2, 7, 1, 1, 11):                                    # one sequence in portions
        rs = recurrent([0, size], [2], [1 if a == 0 else 0], state, dev)
        gx, gh, ghs = lops.stream_norm(pad(x[a:a + size], F32), width, eps, pad(y[a:a + size], dt), *args, rs, 0)
        close(gx[:, :width], xs[a:a + size], F32)
        close(gh[:, :width], h[a:a + size], dt)
        close(ghs[:, :width], hs[a:a + size], dt)
        assert not gh[:, width:].any() and not ghs[:, width:].any()
        close(state[0, 2], h[a + size - 1], F32)
        a += size
    # three sequences in one batch, one of them a padding row
    rs = recurrent([0, 5, 6, 15], [0, -1, 1], [1, 0, 1], state, dev)
    _, _, ghs = lops.stream_norm(pad(x[:15], F32), width, eps, pad(y[:15], dt), *args, rs, 0)
    close(ghs[:5, :width], hs[:5], dt)
    close(ghs[6:15, :width], oracle.token_shift(h[6:15], mix), dt)
    close(state[0, 0], h[4], F32)
    close(state[0, 1], h[14], F32)
    close(state[0, 2], h[22], F32)


@gpu
def test_stream_norm_with_several_rows_per_block():
    n, width = 2700, 96
    x, w, mix = rnd(n, width), rnd(width, seed=3), rnd(width, seed=4)
    h = oracle.grouped_norm(x, w, 2, 1e-5)
    qo = [0, 1, 4, 1300, 1301, 2700]
    state = rnd(1, 5, width, seed=9).cuda()
    before = state.cpu().clone()
    rs = recurrent(qo, [4, 3, 2, 1, 0], [0, 1, 0, 1, 0], state, "cuda")
    _, _, hs = lops.stream_norm(x.cuda(), width, 1e-5, norm_w=w.cuda(), groups=2, shift=mix.cuda(), rs=rs, layer=0)
    for i, (a, b) in enumerate(zip(qo[:-1], qo[1:])):
        prev = torch.cat([torch.zeros(1, width) if rs.reset_host[i] else before[0, 4 - i][None], h[a:b - 1]])
        close(hs[a:b], h[a:b] + (prev - h[a:b]) * mix, F32)
        close(state[0, 4 - i], h[b - 1], F32)


def spec_of(**kw):
    base = dict(heads=3, dim=24, rot_dim=12, vdim=16, kv_rank=40, window=10, scale=0.2, rope_base=50.0, rot_dims=12)
    return LatentSpec(**{**base, **kw})


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("kw", [{}, {"dim": 33, "rot_dim": 6, "rot_dims": 6, "kv_rank": 50}, {"rot_dims": 8},
                                {"heads": 1, "dim": 16, "rot_dim": 16, "rot_dims": 16}])
def test_latent_rows(path, kw):
    dev, dt = path
    s, n = spec_of(**kw), 9
    qkv = rnd(n, s.proj_rows, dtype=dt, std=2)
    pos = torch.tensor([0, 1, 2, 5, 63, 64, 1000, 4095, 7])
    slots = torch.tensor([4, 9, 0, 31, 17, 2, -1, 30, 16], dtype=torch.int32)
    nw = rnd(s.kv_rank, seed=1, dtype=dt)
    table = s.rotary.frequencies(dev)
    cache = torch.full((2, 16, s.row + 16), 7.0, dtype=dt, device=dev)
    q = lops.latent_rows(qkv.to(dev, dt), pos.to(dev, torch.int32), slots.to(dev), table, nw.to(dev, dt), cache, s, 1e-5, s.row,
                         s.rank_pad, copy_nope=False)

    def turn(x):
        return torch.cat([oracle.rotate(x[..., :s.rot_dims], pos, s.rope_base), x[..., s.rot_dims:]], -1)
    qs = qkv[:, :s.q_rows].reshape(n, s.heads, s.qk_dim)
    close(q[..., s.rank_pad:s.rank_pad + s.rot_dim], turn(qs[..., s.dim:]), dt, f32=2e-4)
    assert not q[..., s.rank_pad + s.rot_dim:].any()
    c = oracle.rms(qkv[:, s.q_rows:s.q_rows + s.kv_rank], 1e-5) * nw
    kr = turn(qkv[:, s.q_rows + s.kv_rank:])
    flat = cache.view(32, -1).float().cpu()
    for i, slot in enumerate(slots.tolist()):
        if slot >= 0:
            close(flat[slot, :s.kv_rank], c[i], dt)
            close(flat[slot, s.rank_pad:s.rank_pad + s.rot_dim], kr[i], dt, f32=2e-4)
            assert not flat[slot, s.kv_rank:s.rank_pad].any() and not flat[slot, s.rank_pad + s.rot_dim:].any()
    untouched = [i for i in range(32) if i not in slots.tolist()]
    assert (flat[untouched] == 7.0).all()
    wide = lops.latent_rows(qkv.to(dev, dt), pos.to(dev, torch.int32), slots.to(dev), table, None, None, s, 1e-5, 64, s.dim, copy_nope=True)
    close(wide[..., :s.dim], qs[..., :s.dim], dt)
    close(wide[..., s.dim:s.qk_dim], turn(qs[..., s.dim:]), dt, f32=2e-4)
    assert not wide[..., s.qk_dim:].any()


# ------------------------------------------------------------------ attention over a paged latent cache
def paged(c, kr, s, page, dt, dev, seed=0):
    """Cache rows of one sequence in shuffled pages: (cache, page ids). Other pages hold large values."""
    n = c.shape[0]
    npg = -(-n // page)
    ids = torch.randperm(npg + 3, generator=torch.Generator().manual_seed(seed))[:npg]
    cache = torch.full((npg + 4, page, s.row), 30.0)
    rows = torch.zeros(npg * page, s.row)
    rows[:n, :s.kv_rank], rows[:n, s.rank_pad:s.rank_pad + s.rot_dim] = c, kr
    cache[ids] = rows.view(npg, page, s.row)
    cache[-1] = 0
    return cache.to(dev, dt), ids.tolist()


def plans(qlen, kv, ids, page, window, dev, s):
    t = lambda a: torch.from_numpy(np.ascontiguousarray(a, np.int32)).to(dev)
    qo, ptr_ = np.array([0, qlen]), np.array([0, len(ids)])
    host = ops.AttnBatch(qo, ptr_, np.asarray(ids), np.array([kv]), None, window - 1)
    if dev == "cpu":
        return host
    if qlen == 1:
        ir, st, en, ip, ci = ops.plan_even_items(np.array([kv]), 3, 64, window - 1, min_keys=32)
        scratch = torch.empty(ops.decode_scratch_floats(64, s.heads, s.row), device=dev)
        return ops.DecodePlan(t(ids), t(ptr_), t(ir), t(st), t(en), t(ip), t([len(ir)]), scratch, 64, 1, 3, page, window - 1,
                              kv_lens=t([kv]), cta_items=t(ci))
    tr, tq = ops.plan_prefill_tiles(qo, 1, 256, [kv])
    return ops.PrefillPlan(t(ids), t(ptr_), t(qo), t([kv]), t(tr), t(tq), len(tr), page, window_left=window - 1, tile_rows=256, host=host)


def attention_oracle(q_lat, q_rot, c, kr, s, first):
    """q_* of the last tokens, c / kr of all: weighted latents per head, token `first` + i against its window."""
    out = []
    for h in range(s.heads):
        sc = torch.full((c.shape[0], c.shape[0]), 0.0)
        sc[first:] = (q_lat[:, h] @ c.t() + q_rot[:, h] @ kr.t()) * s.scale
        out.append((oracle.windowed_softmax(sc, s.window) @ c)[first:])
    return torch.stack(out, 1)


SHAPES = [{}, {"heads": 1, "kv_rank": 16, "rot_dim": 2, "rot_dims": 2}, {"heads": 20, "kv_rank": 130}, {"heads": 33, "kv_rank": 64},
          {"heads": 5, "kv_rank": 300, "rot_dim": 64, "rot_dims": 64}, {"heads": 70, "kv_rank": 32}, {"heads": 2, "kv_rank": 600}]


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("kw", SHAPES)
def test_latent_attention_sees_its_window_and_no_more(path, kw):
    """One key stands out in every head's scores and carries a latent of its own; it is placed just inside and just outside
    the window, at page and tile borders, for a decoded token and for a prompt's portion of two tokens and more."""
    dev, dt = path
    page = 16
    for window, kv in ((10, 40), (64, 129), (65, 200), (300, 290), (1, 17)):
        s = spec_of(window=window, **kw)
        for qlen in (1, 2, 19) if kv > 19 else (1, 2):
            first = kv - qlen
            for gap in sorted({0, window - 1, window, 15, 16, 63, 64, first} & set(range(first + 1))):
                at = first - gap                    # the key that stands out, `gap` before the portion's first token
                c, kr = rnd(kv, s.kv_rank, dtype=dt, std=0.3), rnd(kv, s.rot_dim, seed=1, dtype=dt)
                c[at] = rnd(s.kv_rank, seed=7, dtype=dt, std=2)
                q_lat = (c[at] / c[at].norm() * (12 / s.scale / c[at].norm()))[None, None].expand(qlen, s.heads, -1) \
                    + rnd(qlen, s.heads, s.kv_rank, seed=2, std=0.2)
                q_lat, q_rot = q_lat.to(dt).float(), rnd(qlen, s.heads, s.rot_dim, seed=3, dtype=dt)
                cache, ids = paged(c, kr, s, page, dt, dev)
                q = torch.zeros(qlen, s.heads, s.row)
                q[..., :s.kv_rank], q[..., s.rank_pad:s.rank_pad + s.rot_dim] = q_lat, q_rot
                rs = recurrent([0, qlen], [0], [0], torch.zeros(1, 1, 8, device=dev), dev)
                slots = torch.zeros(qlen, dtype=torch.int32, device=dev)
                got = lops.latent_attention(q.to(dev, dt), cache, plans(qlen, kv, ids, page, window, dev, s), rs, slots, s, page, window - 1)
                ref = attention_oracle(q_lat, q_rot, c, kr, s, first)
                close(got[..., :s.kv_rank], ref, dt, f32=2e-4, bf16=2e-2)


@gpu
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("heads,rank", [(20, 48), (40, 256), (3, 320), (33, 130)])
def test_decode_batch_cut_over_ctas_under_layers_of_unequal_windows(heads, rank, dtype):
    """One plan for the widest layer, cut so that requests are split and CTAs have several items; a layer with a narrower
    window sees nothing of some items. Padding requests at the end have no items."""
    kvs, page = [1, 40, 300, 700, 129, 16, 17, 128], 16
    plan_window, r = 600, len(kvs)
    s0 = spec_of(heads=heads, kv_rank=rank, scale=0.3)
    cs = [rnd(k, rank, seed=10 + i, dtype=dtype, std=0.5) for i, k in enumerate(kvs)]
    krs = [rnd(k, s0.rot_dim, seed=30 + i, dtype=dtype) for i, k in enumerate(kvs)]
    caches, ids, ptr_, base = [], [], [0], 0
    for c, kr in zip(cs, krs):
        cache, pid = paged(c, kr, s0, page, dtype, "cpu", seed=len(ids))
        caches.append(cache[:-1])
        ids += [x + base for x in pid]
        base += len(cache) - 1
        ptr_.append(len(ids))
    cache = torch.cat(caches + [torch.zeros(1, page, s0.row)]).to("cuda", dtype)
    q = torch.zeros(r + 2, heads, s0.row)
    q[..., :rank] = rnd(r + 2, heads, rank, seed=1, dtype=dtype)
    q[..., s0.rank_pad:s0.rank_pad + s0.rot_dim] = rnd(r + 2, heads, s0.rot_dim, seed=2, dtype=dtype)
    t = lambda a: torch.from_numpy(np.ascontiguousarray(a, np.int32)).cuda()
    for ctas in (1, 3, 11):
        ir, st, en, ip, ci = ops.plan_even_items(np.array(kvs), ctas, 64, plan_window - 1, min_keys=32)
        pad = lambda a: np.concatenate([a, [a[-1]] * 2])
        plan = ops.DecodePlan(t(ids), t(pad(np.array(ptr_))), t(ir), t(st), t(en), t(pad(ip)), t([len(ir)]),
                              torch.full((ops.decode_scratch_floats(64, heads, s0.row),), float("nan"), device="cuda"), 64, r + 2, ctas,
                              page, plan_window - 1, kv_lens=t(kvs + [0, 0]), cta_items=t(ci))
        rs = recurrent(list(range(r + 3)), list(range(r)) + [-1, -1], [0] * (r + 2), torch.zeros(1, r, 8, device="cuda"), "cuda")
        slots = t([0] * r + [-1, -1])
        for window in (600, 100, 7, 1):
            s = spec_of(heads=heads, kv_rank=rank, scale=0.3, window=window)
            got = lops.latent_attention(q.to("cuda", dtype), cache, plan, rs, slots, s, page, window - 1)
            for i, k in enumerate(kvs):
                ref = attention_oracle(q[i:i + 1, :, :rank], q[i:i + 1, :, s.rank_pad:s.rank_pad + s.rot_dim], cs[i], krs[i], s, k - 1)
                close(got[i:i + 1, :, :rank], ref, dtype, f32=2e-4, bf16=2e-2)
    ops.check_kernel_status()


@gpu
@pytest.mark.parametrize("dims", [(24, 12, 16), (96, 32, 128), (50, 14, 64), (16, 16, 8), (100, 20, 40)])
def test_projected_prefill(dims):
    """Prefill on projected keys and values: unequal requests, cached pasts, windows that start inside a page."""
    dim, rot, vdim = dims
    for window, page in ((37, 16), (130, 32), (1000, 16)):
        s = spec_of(heads=3, dim=dim, rot_dim=rot, rot_dims=rot, vdim=vdim, kv_rank=48, window=window, scale=(dim + rot) ** -0.5)
        d = lops.projected_width(s)
        uk, uv = rnd(s.heads * dim, 48, dtype=BF16, std=0.3), rnd(s.heads * vdim, 48, seed=1, dtype=BF16, std=0.3)
        w = torch.zeros(s.heads, 2, d, s.row)
        w[:, 0, :dim, :48], w[:, 1, :vdim, :48] = uk.view(s.heads, dim, 48), uv.view(s.heads, vdim, 48)
        w[:, 0, dim:dim + rot, s.rank_pad:s.rank_pad + rot] = torch.eye(rot)
        qlens, kvs = [130, 2, 300, 1], [130, 171, 420, 77]
        caches, ids, ptr_, refs, qs = [], [], [0], [], []
        base = 0
        for i, (ql, kv) in enumerate(zip(qlens, kvs)):
            c, kr = rnd(kv, 48, seed=10 + i, dtype=BF16), rnd(kv, rot, seed=20 + i, dtype=BF16)
            cache, pid = paged(c, kr, s, page, BF16, "cpu", seed=i)
            caches.append(cache[:-1])
            ids += [p + base for p in pid]
            base += len(cache) - 1
            ptr_.append(len(ids))
            q = rnd(ql, s.heads, dim + rot, seed=30 + i, dtype=BF16, std=2)
            qs.append(torch.nn.functional.pad(q, (0, d - dim - rot)))
            out = []
            for h in range(s.heads):
                k = torch.cat([(c @ uk[h * dim:(h + 1) * dim].t()).to(BF16).float(), kr], 1)
                sc = torch.zeros(kv, kv)
                sc[kv - ql:] = q[:, h] @ k.t() * s.scale
                out.append((oracle.windowed_softmax(sc, window) @ (c @ uv[h * vdim:(h + 1) * vdim].t()))[kv - ql:])
            refs.append(torch.cat(out, 1))
        t = lambda a: torch.from_numpy(np.ascontiguousarray(a, np.int32)).cuda()
        qo = np.concatenate([[0], np.cumsum(qlens)])
        tr, tq = ops.plan_prefill_tiles(qo, 1, 256, kvs)
        plan = ops.PrefillPlan(t(ids), t(ptr_), t(qo), t(kvs), t(tr), t(tq), len(tr), page, window_left=window - 1, tile_rows=256,
                               host=ops.AttnBatch(qo, np.asarray(ptr_), np.asarray(ids), np.asarray(kvs)))
        cache = torch.cat(caches + [torch.zeros(1, page, s.row)]).to("cuda", BF16)
        wide = torch.full((int(qo[-1]), s.heads * vdim + 8), 5.0, dtype=BF16, device="cuda")
        out = lops.projected_prefill_attention(torch.cat(qs).to("cuda", BF16), cache, plan, w.view(-1, s.row).to("cuda", BF16), s, page,
                                               window - 1, wide[:, :s.heads * vdim])
        close(out, torch.cat(refs), BF16, bf16=2e-2)
        assert (wide[:, s.heads * vdim:] == 5.0).all()
        ops.check_kernel_status()


# ------------------------------------------------------------------ products and activations
@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("n,heads,k,m", [(3, 4, 24, 40), (70, 3, 33, 21), (1, 1, 256, 130), (130, 2, 7, 1)])
def test_per_head(path, n, heads, k, m):
    dev, dt = path
    x, w = rnd(n, heads, k + 5, dtype=dt), rnd(heads, m, k, seed=1, dtype=dt)
    out = torch.full((n, heads * m + 3), 9.0, dtype=dt, device=dev)
    lops.per_head(x.to(dev, dt)[..., :k], w.to(dev, dt), out[:, :heads * m].view(n, heads, m) if out.stride(0) == heads * m
                  else out.as_strided((n, heads, m), (out.stride(0), m, 1)))
    close(out[:, :heads * m], torch.einsum("nhk,hmk->nhm", x[..., :k], w).reshape(n, -1), dt)
    assert (out[:, heads * m:] == 9.0).all()


@pytest.mark.parametrize("path", PATHS)
def test_xielu_gate_and_stream_add(path):
    dev, dt = path
    y, b, act = rnd(5, 37, dtype=dt, std=4), rnd(37, seed=1, dtype=dt), torch.tensor([0.7, -1.3]).to(dt).float()
    wide = torch.zeros(5, 50, dtype=dt, device=dev)
    wide[:, 6:43] = y.to(dev, dt)
    lops.bias_xielu(wide[:, 6:43], b.to(dev, dt), act.to(dev, dt))
    close(wide[:, 6:43], oracle.xielu(y + b, act[0], act[1]), dt)
    x, d = rnd(5, 40, seed=2), rnd(5, 40, seed=3, dtype=dt)
    nx, cp = lops.stream_add(x.to(dev), d.to(dev, dt), None, copy=True)
    close(nx, x + d, F32)
    close(cp, x + d, dt)
    z, table = rnd(6, 16, seed=4, dtype=dt, std=2), rnd(11, 30, seed=5, dtype=dt)
    toks = torch.tensor([3, 0, 10, 10, 1, 7], dtype=torch.int32)
    g = lops.side_gate(z.to(dev, dt), table.to(dev, dt), toks.to(dev), 20, 10)
    close(g[:, :10], oracle.gelu_tanh(z[:, :10]) * table[toks.long(), 20:30], dt)
    assert not g[:, 10:].any()


@gpu
@pytest.mark.parametrize("m", [1, 5, 64, 65, 128, 130, 515, 4096])
@pytest.mark.parametrize("n,k", [(40, 24), (320, 104), (1344, 4096), (4096, 1032)])
def test_gemm_epilogues(m, n, k):
    """xIELU with bias, and the 32-bit stream with bias and its bf16 copy; outputs as column ranges; every launch shape
    (whole tiles, swapped operands, split K, CTA pairs)."""
    x, w, b = rnd(m, k, dtype=BF16), rnd(n, k, seed=1, dtype=BF16, std=k ** -0.5), rnd(n, seed=2, dtype=BF16)
    act = torch.tensor([0.4, -0.8]).to(BF16)
    z = (x.double() @ w.double().t() + b.double()).float()
    wide = torch.full((m, n + 16), 3.0, dtype=BF16, device="cuda")
    lops.gemm_xielu(x.to("cuda", BF16), w.to("cuda", BF16), b.to("cuda", BF16), act.cuda(), wide[:, 8:8 + n])
    close(wide[:, 8:8 + n], oracle.xielu(z, act[0].float(), act[1].float()), BF16)
    assert (wide[:, :8] == 3.0).all() and (wide[:, 8 + n:] == 3.0).all()
    s = rnd(m, n, seed=3)
    for copy in (True, False):
        sx, cp = lops.gemm_stream(x.to("cuda", BF16), w.to("cuda", BF16), b.to("cuda", BF16), s.cuda(), copy=copy)
        close(sx, s + z, F32)
        if copy:
            close(cp, s + z, BF16)
    ops.check_kernel_status()


@gpu
@pytest.mark.parametrize("n", [1, 64, 100, 700])
def test_split_product_with_its_gate(n):
    x, w = rnd(n, 1000, dtype=BF16), rnd(24, 1000, seed=1, dtype=BF16, std=0.03)
    table, toks = rnd(9, 60, seed=2, dtype=BF16), torch.arange(n, dtype=torch.int32) % 9
    z = lops.split_product(x.to("cuda", BF16), w.to("cuda", BF16))
    close(z.sum(0), x @ w.t(), F32, f32=1e-4)
    g = lops.side_gate(z, table.to("cuda", BF16), toks.cuda(), 30, 20)
    close(g[:, :20], oracle.gelu_tanh(x @ w.t())[:, :20] * table[toks.long(), 30:50], BF16)
    assert not g[:, 20:].any()


@pytest.mark.parametrize("path", PATHS)
def test_stream_embed(path):
    dev, dt = path
    table = rnd(13, 20, dtype=dt)
    x = lops.stream_embed(torch.tensor([12, 0, 5], dtype=torch.int32, device=dev), table.to(dev, dt), 24)
    assert torch.equal(x[:, :20].cpu(), table[[12, 0, 5]]) and not x[:, 20:].any()
