"""Retodra through the driver, the context manager and the engine, against the plain statement in retodra_oracle.py: whole
prompts, token by token, portions, unequal batches, pages and state slots used again, window edges, long decoding, greedy
generation. Each runs on the CPU path (32-bit) and, on a GPU, on the kernels in 32-bit and in bf16."""
import json

import numpy as np
import pytest
import retodra_models as rm
import retodra_oracle as oracle
import torch

from pie_b200.driver.executor import TorchDriver
from pie_b200.inferlets import install_all
from pie_b200.models import loader
from pie_b200.models.block_spec import ExpertsSpec, GatedLinearSpec, ParallelSpec
from pie_b200.models.config import ModelConfig, preset
from pie_b200.runtime.engine import Engine, EngineConfig
from pie_b200.runtime.rs_cache import RsState
from pie_b200.runtime.tokenizer import ByteTokenizer
from pie_b200.runtime.trace import Replay

PATHS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
# root mean square of the difference over the vocabulary, against the root mean square of the logits
LIMIT = {"float32": 3e-5, "bfloat16": 0.04}
STEP = {"float32": 0.2, "bfloat16": 1.0}        # see retodra_models.tensors
_WANT: dict = {}


def want(name, n, seed=0, dtype="float32"):
    """Oracle logits of every position of the prompt (name, n, seed), with the weights that runs in `dtype` take."""
    key = (name, n, seed, STEP[dtype])
    if key not in _WANT:
        cfg = rm.CONFIGS[name]
        _WANT[key] = oracle.forward(cfg, rm.tensors(cfg, step=STEP[dtype]), rm.prompt(cfg, n, seed)).numpy()
    return _WANT[key]


def error(got, ref):
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def load(cfg_d, t, device, dtype):
    cfg, reader = ModelConfig.from_hf(cfg_d), loader.TensorDictReader(t)
    loader.complete_blocks(cfg, reader)
    return cfg, loader.execute_program(loader.compile_program(cfg, list(t), dtype=dtype), reader, device)


def make_driver(name, path, pages=40, slots=4, max_tokens=512, **kw):
    device, dtype = path
    cfg, w = load(rm.CONFIGS[name], rm.tensors(rm.CONFIGS[name], step=STEP[dtype]), device, dtype)
    return TorchDriver(cfg, device, weights=w, num_pages=pages, page_size=kw.pop("page_size", 16), max_requests=slots,
                       max_tokens=max_tokens, rs_slots=slots, compute_dtype=dtype, **kw)


def entry(rid, toks, a, b):
    return {"id": rid, "tokens": toks[a:b], "want": list(range(b - a))}


def run_cuts(rp, rid, toks, cuts):
    """Logits of every position, the prompt cut at `cuts`."""
    edges = [0, *cuts, len(toks)]
    return np.concatenate([rp.step([entry(rid, toks, a, b)], [rid] if b == len(toks) else [])
                           for a, b in zip(edges[:-1], edges[1:])])


def close(got, ref, dtype):
    """Sharp attention now and then turns a rounding into more (two keys with almost the same score): one position in fifty
    may be over the limit, none over three times it."""
    e = error(got, ref)
    assert e.max() <= 3 * LIMIT[dtype] and (e > LIMIT[dtype]).sum() <= max(1, len(e) // 50), (float(e.max()), int(e.argmax()))


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", list(rm.CONFIGS))
def test_whole_prompt_token_by_token_and_portions(name, path):
    n = 50 if path[0] == "cpu" else 200
    cfg = rm.CONFIGS[name]
    toks, ref = rm.prompt(cfg, n), want(name, n, dtype=path[1])
    rp = Replay(make_driver(name, path))
    close(run_cuts(rp, "a", toks, []), ref, path[1])
    close(run_cuts(rp, "b", toks, list(range(1, n))), ref, path[1])
    for i, size in enumerate((2, 3, 16, 29)):
        close(run_cuts(rp, f"c{i}", toks, list(range(size, n, size))), ref, path[1])
    # a prompt, then single tokens, then a portion again, ending at and next to page borders
    close(run_cuts(rp, "d", toks, [15, 16, 17, 31, 32, 47, n - 2]), ref, path[1])
    assert rp.driver.rs.num_slots == 4 and rp.contexts.rs[0].slot_of == {}
    rp.contexts.audit()


@pytest.mark.parametrize("path", PATHS)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_unequal_batches_against_each_alone_with_pages_and_slots_reused(name, path):
    """Four live requests of unequal lengths in every step: portions beside single tokens, requests left out of steps,
    ended and replaced; the pool holds little more than the live tokens, so pages and slots change hands."""
    cfg = rm.CONFIGS[name]
    lens = [33, 50, 7, 64, 40, 18, 55, 1, 30]
    if path[0] != "cpu":
        lens[3] = 150                                   # several 64-token pieces and key blocks beside short portions
    prompts = [rm.prompt(cfg, n, i) for i, n in enumerate(lens)]
    rng = np.random.default_rng(5)
    drv = make_driver(name, path, pages=22)
    rp, at, live, waiting = Replay(drv), {}, [], list(range(len(lens)))
    got = {i: [] for i in range(len(lens))}
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries = []
        for i in [x for x in live if len(live) == 1 or rng.random() < 0.8] or live[:1]:
            k = min(int(rng.choice([1, 1, 2, 5, 17, 31, 90])), lens[i] - at[i])
            entries.append((i, at[i], at[i] + k))
            at[i] += k
        entries = [entries[j] for j in rng.permutation(len(entries))]
        end = [i for i, _, b in entries if b == lens[i]]
        rows = rp.step([entry(f"r{i}", prompts[i], a, b) for i, a, b in entries], [f"r{i}" for i in end])
        o = 0
        for i, a, b in entries:
            got[i].append(rows[o:o + b - a])
            o += b - a
        live = [i for i in live if i not in end]
    for i in range(len(lens)):
        close(np.concatenate(got[i]), want(name, lens[i], i, path[1]), path[1])
    assert rp.contexts.pages_used() == 0


@pytest.mark.parametrize("path", PATHS)
def test_long_decoding_and_large_pages(path):
    n = 120 if path[0] == "cpu" else 330
    for name, page in (("mixed", 16), ("odd", 32), ("wide", 64)):
        toks = rm.prompt(rm.CONFIGS[name], n)
        rp = Replay(make_driver(name, path, page_size=page), page)
        close(run_cuts(rp, "a", toks, list(range(20, n))), want(name, n, dtype=path[1]), path[1])
        close(run_cuts(rp, "b", toks, [90]), want(name, n, dtype=path[1]), path[1])


@pytest.mark.parametrize("path", PATHS)
def test_padded_buckets_do_not_touch_the_state(path):
    """Three single-token requests run in a bucket of four; a fourth request left out meanwhile goes on unharmed."""
    cfg = rm.CONFIGS["mixed"]
    prompts = [rm.prompt(cfg, 24, i) for i in range(4)]
    rp = Replay(make_driver("mixed", path))
    rows = [[r] for r in np.split(rp.step([entry(f"r{i}", prompts[i], 0, 9) for i in range(4)]), 4)]
    for s in range(9, 24):
        ids = [0, 1, 2] if s < 16 else [0, 1, 2, 3]
        spans = [(i, s if i < 3 else s - 7) for i in ids]
        out = rp.step([entry(f"r{i}", prompts[i], a, a + 1) for i, a in spans])
        for (i, _), r in zip(spans, out):
            rows[i].append(r[None])
    for i in range(4):
        got = np.concatenate(rows[i])
        close(got, want("mixed", 24, i, path[1])[:len(got)], path[1])


@pytest.mark.gpu
def test_graphs_of_small_batches_survive_larger_ones():
    """Expert scratch grows with the batch; a decode graph captured before that goes on working on its own."""
    drv = make_driver("mixed", ("cuda", "bfloat16"))
    rp, toks = Replay(drv), rm.prompt(rm.CONFIGS["mixed"], 200)
    a = [rp.step([entry("a", toks, i, i + 1)]) for i in range(6)]
    rp.step([entry("b", toks, 0, 200)], ["b"])
    a += [rp.step([entry("a", toks, i, i + 1)]) for i in range(6, 20)]
    close(np.concatenate(a), want("mixed", 200, dtype="bfloat16")[:20], "bfloat16")
    assert drv.stats["graph_replays"] == 20


def sensitivity(kind):
    """Relative change of the logits when the plain statement itself is wrong in one way."""
    cfg = json.loads(json.dumps(rm.CONFIGS["mixed"]))
    t, toks = rm.tensors(cfg), rm.prompt(cfg, 110)
    good = oracle.forward(cfg, t, toks)
    save = {}

    def swap(name, fn):
        save[name] = getattr(oracle, name)
        setattr(oracle, name, fn)
    state, bucket, rms = oracle.decayed_state, oracle.distance_bucket, oracle.rms
    pars = [s["mixer"] for s in cfg["layers"] if s["type"] == "parallel"]
    if kind in ("window+1", "window-1"):
        for m in pars:
            m["left"]["mask"]["size"] += 1 if kind == "window+1" else -1
    elif kind == "state lost at 60":
        swap("decayed_state", lambda q, k, v, a: torch.cat([state(q[:60], k[:60], v[:60], a[:60]), state(q[60:], k[60:], v[60:], a[60:])]))
    elif kind == "decay after the update":
        swap("decayed_state", lambda q, k, v, a: state(q, k * a, v, a))
    elif kind == "bucket one late":
        swap("distance_bucket", lambda n, b, far: bucket(max(n - 1, 0), b, far))
    elif kind == "no cap":
        swap("softcap", lambda s, cap: s)
    elif kind == "gain not about one":
        swap("norm_about_one", lambda x, w, eps: rms(x, eps) * w)
    elif kind == "choice without correction":
        swap("route", lambda h, r, c, top: oracle_route(h, r, 0 * c, top))
    elif kind == "weights with correction":
        swap("route", lambda h, r, c, top: (oracle_route(h, r, c, top)[0], torch.topk(torch.softmax(h @ r.t(), -1) + c, top).values))
    elif kind == "identity is nothing":
        swap("identity_expert", torch.zeros_like)
    elif kind == "limit":
        swap("clamped_expert", lambda h, w, limit: save["clamped_expert"](h, w, 1.1 * limit))
    elif kind == "sides swapped":
        for m in pars:
            m["left_scale"], m["right_scale"] = m["right_scale"], m["left_scale"]
    elif kind == "no layer scale":
        t = {k: torch.ones_like(v) if ".ls" in k else v for k, v in t.items()}
    try:
        bad = oracle.forward(cfg, t, toks)
    finally:
        for k, v in save.items():
            setattr(oracle, k, v)
    return error(bad.numpy(), good.numpy())[60:].max()


oracle_route = oracle.route


@pytest.mark.parametrize("kind", ["window+1", "window-1", "state lost at 60", "decay after the update", "bucket one late", "no cap",
                                  "gain not about one", "choice without correction", "weights with correction", "identity is nothing",
                                  "limit", "sides swapped", "no layer scale"])
def test_the_models_show_mistakes(kind):
    """A mistake planted in the plain statement moves the logits well past the tolerance of the comparisons."""
    assert sensitivity(kind) > (1.5 if kind == "limit" else 3) * LIMIT["bfloat16"]


# ------------------------------------------------------------------ configuration, loading, engine
def test_configuration_and_registry():
    cfg = ModelConfig.from_hf(rm.CONFIGS["mixed"])
    assert cfg.model_type == "retodra" and cfg.stream32 and cfg.recurrent_layers == [0, 1, 2, 3]
    assert [type(b.mixer) for b in cfg.blocks] == [GatedLinearSpec, ParallelSpec] * 2
    assert cfg.kv_layers == [(2, 64), (4, 64)] and cfg.plan_window_left == 69 and cfg.layer_window_left(1) == 36
    assert cfg.blocks[1].attention.group_pad == 4 and isinstance(cfg.blocks[1].ff, ExpertsSpec) and cfg.blocks[1].ff.outputs == 8
    assert ModelConfig.from_hf(rm.CONFIGS["odd"]).blocks[2].ff is None
    assert ModelConfig.from_hf(rm.CONFIGS["linear"]).kv_elems_per_page(16) == 0
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]),
                   lambda c: c["layers"][1]["mlp"]["router"].update(top=9), lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0)):
        bad = json.loads(json.dumps(rm.CONFIGS["mixed"]))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)
    assert preset("retodra-19b", num_hidden_layers=2).num_hidden_layers == 2


@pytest.mark.parametrize("rows,far", [(12, 90), (8, 64), (32, 128), (2, 9), (16, 1000)])
def test_distance_buckets(rows, far):
    a = ModelConfig.from_hf(rm.CONFIGS["mixed"]).blocks[1].attention
    a.buckets, a.bias_max = rows, far
    got = [a.bucket(n) for n in range(2 * far)]
    assert got == [oracle.distance_bucket(n, rows, far) for n in range(2 * far)]
    assert got[:rows // 2] == list(range(rows // 2)) and got[-1] == rows - 1 and got == sorted(got)


@pytest.mark.parametrize("name", ["mixed", "odd", "ones"])
def test_checkpoint_round_trip_and_type_check(tmp_path, name):
    cfg_d = rm.CONFIGS[name]
    t = rm.tensors(cfg_d)
    cfg, w = loader.load_checkpoint(rm.write_checkpoint(tmp_path / "a", cfg_d, t), "cpu", dtype="bfloat16")
    assert all(b.mixer.rank == rm.ranks(i) for i, b in enumerate(cfg.blocks) if isinstance(b.mixer, GatedLinearSpec))
    loader.export_hf_checkpoint(cfg, w, tmp_path / "b")
    from safetensors.torch import load_file
    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    again, _ = loader.load_checkpoint(tmp_path / "b", "cpu")
    assert again.blocks == cfg.blocks and again.embed_scale == cfg.embed_scale
    key = next(k for k in t if k.endswith("mix.right.o" if name != "linear" else "mix.o"))
    t[key] = t[key][:-1]
    with pytest.raises(loader.LoaderTypeError, match=key):
        loader.load_checkpoint(rm.write_checkpoint(tmp_path / "c", cfg_d, t), "cpu")


def oracle_greedy(name, toks, n):
    cfg, toks = rm.CONFIGS[name], list(toks)
    k = len(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, rm.tensors(cfg), toks)[-1].argmax()))
    return toks[k:]


@pytest.mark.parametrize("path", PATHS[:2])
def test_greedy_generation_through_the_engine(path):
    """Entry point, scheduler, chunked prefill (the prompt exceeds a pass), more contexts than state slots; fork and a lost
    state that is rebuilt from the lineage."""
    name = "mixed"
    drv = make_driver(name, path, pages=64, slots=8, max_tokens=48)
    drv.rs.num_slots = 3
    e = Engine(EngineConfig())
    e.add_model("m", drv, tokenizer=ByteTokenizer(rm.CONFIGS[name]["vocab"]))
    install_all(e)
    try:
        prompts = [rm.prompt(rm.CONFIGS[name], n, i) for i, n in enumerate((70, 9, 30, 50))]
        pids = [e.launch("text-completion", {"prompt_tokens": p, "max_tokens": 5, "temperature": 0.0, "stop_tokens": []})
                for p in prompts]
        outs = [json.loads(e.wait(p, 300))["tokens"] for p in pids]
        assert outs == [oracle_greedy(name, p, 5) for p in prompts]
        from pie_b200.sdk import Context, Model, Sampler

        async def prog(args):
            ctx = Context(Model.load("m"))
            ctx.append(prompts[2])
            first = await ctx.generate(Sampler.argmax(), max_tokens=2).stop([]).collect_tokens()
            child = ctx.fork()
            a = await child.generate(Sampler.argmax(), max_tokens=3).stop([]).collect_tokens()
            ctx._entry.ctxm.rs[0].invalidate(ctx.id)
            b = await ctx.generate(Sampler.argmax(), max_tokens=3).stop([]).collect_tokens()
            state = ctx._entry.ctxm.rs[0].state_of(ctx.id).name
            child.release()
            ctx.release()
            return json.dumps([first, a, b, state])
        e.register_program("t", prog)
        first, a, b, state = json.loads(e.run("t", {}, 300))
        assert first + a == outs[2] and first + b == outs[2] and state == RsState.RESIDENT.name
        assert e.models["m"].ctxm.rs[0].slot_of == {}
    finally:
        e.shutdown()


@pytest.mark.gpu
def test_memory_is_planned_beside_the_states():
    """Pages, passes and state slots from what the device has left; the model then runs."""
    cfg = preset("tiny-retodra")
    drv = TorchDriver(cfg, "cuda", num_pages=0, max_requests=8, max_tokens=512, gpu_mem_utilization=0.3)
    assert drv.rs.num_slots == 16 and drv.kv.num_pages >= 64 and drv.memory_plan.arena_bytes > 0
    rp, toks = Replay(drv), list(range(1, 130))
    a = run_cuts(rp, "a", toks, [])
    assert error(run_cuts(rp, "b", toks, [60, 100, 128]), a).max() < 0.03


def test_bytes_of_pages_and_slots():
    from pie_b200.driver import memory_planner as mp
    from pie_b200.driver.recurrent import RecurrentStateCache
    cfg = ModelConfig.from_hf(rm.CONFIGS["mixed"])
    assert mp.kv_bytes_per_page(cfg, 16) == 2 * 16 * 2 * (2 * 64 + 4 * 64)
    rs = RecurrentStateCache(cfg, 3, "cpu")
    assert rs.bytes_per_slot == 4 * (3 * 24 * 40 + 2 * 16 * 24 + 2 * 48 * 24 + 5 * 24 * 8)
    rs.linear_state[1] = torch.arange(rs.linear_state.shape[1])
    rs.copy_slot(1, 2)
    assert torch.equal(rs.linear_state[1], rs.linear_state[2]) and not rs.linear_state[0].any()
    assert mp.arena_bytes(cfg, 1024, 8) > 1024 * 96 * 16


def test_swap_copies_pages_of_unequal_layers():
    from pie_b200.driver.kv_cache import KVCache
    from pie_b200.driver.schema import CopyDir, CopyRequest
    kv = KVCache(0, 4, 1, 16, 64, torch.float32, "cpu", swap_pages=2, layer_shapes=[((2, 2, 16, 64), None), ((2, 4, 16, 128), None)])
    for i, t in enumerate(kv.parts):
        t[:, 1] = 7.0 + i
    assert kv.page_bytes_all_layers == 2 * 16 * (2 * 64 + 4 * 128) * 4
    kv.copy(CopyRequest(CopyDir.D2H, np.array([1]), np.array([0])))
    kv.copy(CopyRequest(CopyDir.H2H, np.array([0]), np.array([1])))
    kv.copy(CopyRequest(CopyDir.H2D, np.array([1]), np.array([3])))
    kv.copy(CopyRequest(CopyDir.D2D, np.array([3]), np.array([2])))
    assert all(bool((kv.data[i][2] == 7.0 + i).all()) and not kv.data[i][0].any() for i in range(2))
