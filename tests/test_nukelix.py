"""Nukelix through the driver, the context manager and the engine, against the plain statement in nukelix_oracle.py: whole
prompts, token by token, portions, unequal batches, pages and state slots used again, edges of windows and of the kept first
tokens, long decoding, greedy generation. Each runs on the CPU path (32-bit) and, on a GPU, on the kernels in 32-bit and in
bf16."""
import json

import numpy as np
import nukelix_models as nm
import nukelix_oracle as oracle
import pytest
import torch

from pie_b200.driver.executor import TorchDriver
from pie_b200.inferlets import install_all
from pie_b200.models import loader
from pie_b200.models.block_spec import GroupedAttentionSpec, LatentSpec, MatrixMemorySpec, ParallelSpec
from pie_b200.models.config import ModelConfig, preset
from pie_b200.runtime.engine import Engine, EngineConfig
from pie_b200.runtime.rs_cache import RsState
from pie_b200.runtime.tokenizer import ByteTokenizer
from pie_b200.runtime.trace import Replay

PATHS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
# root mean square of the difference over the vocabulary, against the root mean square of the logits
LIMIT = {"float32": 3e-5, "bfloat16": 0.04}
_WANT: dict = {}
_TENSORS: dict = {}


def tensors(name):
    if name not in _TENSORS:
        _TENSORS[name] = nm.tensors(nm.CONFIGS[name])
    return _TENSORS[name]


def want(name, n, seed=0):
    """Oracle logits of every position of the prompt (name, n, seed)."""
    if (name, n, seed) not in _WANT:
        cfg = nm.CONFIGS[name]
        _WANT[name, n, seed] = oracle.forward(cfg, tensors(name), nm.prompt(cfg, n, seed)).numpy()
    return _WANT[name, n, seed]


def error(got, ref):
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def make_driver(name, path, pages=40, slots=4, max_tokens=512, **kw):
    device, dtype = path
    cfg, t = ModelConfig.from_hf(nm.CONFIGS[name]), tensors(name)
    w = loader.execute_program(loader.compile_program(cfg, list(t), dtype=dtype), loader.TensorDictReader(t), device)
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
@pytest.mark.parametrize("name", list(nm.CONFIGS))
def test_whole_prompt_token_by_token_and_portions(name, path):
    n = 50 if path[0] == "cpu" else 200
    toks, ref = nm.prompt(nm.CONFIGS[name], n), want(name, n)
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
    cfg = nm.CONFIGS[name]
    lens = [33, 50, 7, 64, 40, 18, 55, 1, 30]
    if path[0] != "cpu":
        lens[3] = 150                                   # several 64-token pieces and key blocks beside short portions
    prompts = [nm.prompt(cfg, n, i) for i, n in enumerate(lens)]
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
        close(np.concatenate(got[i]), want(name, lens[i], i), path[1])
    assert rp.contexts.pages_used() == 0


@pytest.mark.parametrize("path", PATHS)
def test_long_decoding_and_large_pages(path):
    n = 120 if path[0] == "cpu" else 330
    for name, page in (("mixed", 16), ("odd", 32), ("wide", 64)):
        toks = nm.prompt(nm.CONFIGS[name], n)
        rp = Replay(make_driver(name, path, page_size=page), page)
        close(run_cuts(rp, "a", toks, list(range(20, n))), want(name, n), path[1])
        close(run_cuts(rp, "b", toks, [90]), want(name, n), path[1])


@pytest.mark.parametrize("path", PATHS)
def test_padded_buckets_do_not_touch_the_state(path):
    """Three single-token requests run in a bucket of four; a fourth request left out meanwhile goes on unharmed."""
    cfg = nm.CONFIGS["mixed"]
    prompts = [nm.prompt(cfg, 24, i) for i in range(4)]
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
        close(got, want("mixed", 24, i)[:len(got)], path[1])


@pytest.mark.gpu
def test_graphs_of_small_batches_survive_larger_ones():
    """Expert scratch grows with the batch; a decode graph captured before that goes on working on its own."""
    drv = make_driver("mixed", ("cuda", "bfloat16"))
    rp, toks = Replay(drv), nm.prompt(nm.CONFIGS["mixed"], 200)
    a = [rp.step([entry("a", toks, i, i + 1)]) for i in range(6)]
    rp.step([entry("b", toks, 0, 200)], ["b"])
    a += [rp.step([entry("a", toks, i, i + 1)]) for i in range(6, 20)]
    close(np.concatenate(a), want("mixed", 200)[:20], "bfloat16")
    assert drv.stats["graph_replays"] == 20


def swapped(kind, cfg, t):
    """Plant one mistake in the plain statement (returns {name: replacement}), its configuration or its tensors."""
    o = {k: getattr(oracle, k) for k in dir(oracle)}
    windows = [s["mixer"]["mask"] for s in cfg["layers"] if "mask" in s["mixer"]]
    every = [s["mixer"] for s in cfg["layers"]]
    if kind in ("window+1", "window-1"):
        for m in windows:
            m["size"] += 1 if kind == "window+1" else -1
    elif kind in ("kept+1", "kept-1"):
        for m in windows:
            m["keep_first"] += 1 if kind == "kept+1" else -1
    elif kind == "sides swapped":
        for m in every:
            if "left" in m:
                m["left_scale"], m["right_scale"] = m["right_scale"], m["left_scale"]
    elif kind == "bias left out":
        for k in t:
            if k.endswith((".q.b", ".k.b", ".v.b")):
                t[k] = torch.zeros_like(t[k])
    elif kind == "frequencies unscaled":
        for m in every:
            m.get("rot", {}).pop("scaling", None)
    return {
        "no sink": {"weights_over_keys": lambda s, see, sink: o["weights_over_keys"](s, see, False)},
        "kept tokens moved": {"rotated": lambda x, f, adjacent, factor=1.0, positions=None: o["rotated"](
            x, f, adjacent, factor, torch.arange(x.shape[0]) % 50 if adjacent and x.shape[1] < 5 else positions)},
        "layouts swapped": {"rotated": lambda x, f, adjacent, *a: o["rotated"](x, f, not adjacent, *a)},
        "cos and sin unscaled": {"rotated": lambda x, f, adjacent, factor=1.0, positions=None: o["rotated"](x, f, adjacent, 1.0, positions)},
        "values unmixed": {"mixed_values": lambda v, first, lam: v},
        "values mixed the other way": {"mixed_values": lambda v, first, lam: o["mixed_values"](v, first, 1 - lam)},
        "no head gate": {"head_gate": lambda x, h, g: x},
        "state lost at 60": {"matrix_memory": lambda q, k, v, i, f: (torch.cat([o["matrix_memory"](q[a], k[a], v[a], i[a], f[a])[0]
                                                                                  for a in (slice(0, 60), slice(60, None))]), None)},
        "gates without cap": {"soft_limit": lambda z, cap: z if z.dim() == 2 and z.shape[1] < 8 else o["soft_limit"](z, cap)},
        "gates swapped": {"log_gates": lambda h, w, cap: tuple(reversed(o["log_gates"](h, w, cap)))},
        "logits uncapped": {"soft_limit": lambda z, cap: z if z.shape[1] > 100 else o["soft_limit"](z, cap)},
        "weight on the output": {"weighted_expert": lambda h, c, w: c * o["expert"](h, w)},
        "weights renormalised": {"route": lambda h, r, top: (o["route"](h, r, top)[0], torch.nn.functional.normalize(
            o["route"](h, r, top)[1], p=1, dim=-1))},
        "one expert fewer": {"route": lambda h, r, top: tuple(x[:, :max(1, top - 1)] for x in o["route"](h, r, top))},
    }.get(kind, {})


KINDS = ["window+1", "window-1", "kept+1", "kept-1", "kept tokens moved", "no sink", "layouts swapped", "frequencies unscaled",
         "cos and sin unscaled", "values unmixed", "values mixed the other way", "no head gate", "bias left out", "state lost at 60",
         "gates without cap", "gates swapped", "logits uncapped", "weight on the output", "weights renormalised", "one expert fewer",
         "sides swapped"]


@pytest.mark.parametrize("kind", KINDS)
def test_the_models_show_mistakes(kind, monkeypatch):
    """A mistake planted in the plain statement moves the logits well past the tolerance of the comparisons."""
    cfg, t, toks = json.loads(json.dumps(nm.CONFIGS["mixed"])), dict(tensors("mixed")), nm.prompt(nm.CONFIGS["mixed"], 110)
    good = want("mixed", 110)
    for name, fn in swapped(kind, cfg, t).items():
        monkeypatch.setattr(oracle, name, fn)
    assert error(oracle.forward(cfg, t, toks).numpy(), good)[60:].max() > 2 * LIMIT["bfloat16"]


# ------------------------------------------------------------------ configuration, loading, engine
def test_configuration_and_registry():
    cfg = ModelConfig.from_hf(nm.CONFIGS["mixed"])
    assert cfg.model_type == "nukelix" and cfg.stream32 and cfg.post_norm and cfg.final_softcap == 20.0
    assert [type(b.mixer) for b in cfg.blocks] == [ParallelSpec, GroupedAttentionSpec, LatentSpec, GroupedAttentionSpec, GroupedAttentionSpec,
                                                   ParallelSpec]
    assert [b.recurrent is not None for b in cfg.blocks] == [True, False, False, False, False, True]
    assert isinstance(cfg.blocks[0].recurrent, MatrixMemorySpec) and cfg.blocks[4].ff is None and cfg.blocks[3].ff.shared == 0
    assert cfg.kv_layers == [(2, 64), (2, 64), (0, 64), (2, 64), (4, 64), (4, 64)] and cfg.plan_window_left == -1
    assert [cfg.blocks[i].attention.v_mix for i in (0, 1, 3, 4)] == [False, True, True, False] and cfg.blocks[1].attention.group_pad == 4
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0),
                   lambda c: c["layers"][1]["mlp"]["router"].update(top=9), lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26), lambda c: c["layers"][2]["mixer"]["rot"].update(dims=5),
                   lambda c: c["layers"][3]["mixer"].update(vdim=16)):
        bad = json.loads(json.dumps(nm.CONFIGS["mixed"]))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)
    assert preset("nukelix-20b", num_hidden_layers=3).num_hidden_layers == 3


@pytest.mark.parametrize("name", list(nm.CONFIGS))
def test_checkpoint_round_trip_and_type_check(tmp_path, name):
    cfg_d, t = nm.CONFIGS[name], dict(tensors(name))
    cfg, w = loader.load_checkpoint(nm.write_checkpoint(tmp_path / "a", cfg_d, t), "cpu", dtype="bfloat16")
    loader.export_hf_checkpoint(cfg, w, tmp_path / "b")
    from safetensors.torch import load_file
    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    again, _ = loader.load_checkpoint(tmp_path / "b", "cpu")
    assert again.blocks == cfg.blocks and again.final_softcap == cfg.final_softcap
    key = next(k for k in t if k.endswith(".mlp.router"))
    t[key] = t[key][:-1] if t[key].shape[0] > 1 else t[key][:, :-1]
    with pytest.raises(loader.LoaderTypeError, match=key):
        loader.load_checkpoint(nm.write_checkpoint(tmp_path / "c", cfg_d, t), "cpu")


def oracle_greedy(name, toks, n):
    toks, k = list(toks), len(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(nm.CONFIGS[name], tensors(name), toks)[-1].argmax()))
    return toks[k:]


@pytest.mark.parametrize("path", PATHS[:2])
def test_greedy_generation_through_the_engine(path):
    """Entry point, scheduler, chunked prefill (the prompt exceeds a pass), more contexts than state slots; fork and a lost
    state that is rebuilt from the lineage."""
    name = "mixed"
    drv = make_driver(name, path, pages=64, slots=8, max_tokens=48)
    drv.rs.num_slots = 3
    e = Engine(EngineConfig())
    e.add_model("m", drv, tokenizer=ByteTokenizer(nm.CONFIGS[name]["vocab"]))
    install_all(e)
    try:
        prompts = [nm.prompt(nm.CONFIGS[name], n, i) for i, n in enumerate((70, 9, 30, 50))]
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
    cfg = preset("tiny-nukelix")
    drv = TorchDriver(cfg, "cuda", num_pages=0, max_requests=8, max_tokens=512, gpu_mem_utilization=0.3)
    assert drv.rs.num_slots == 16 and drv.kv.num_pages >= 64 and drv.memory_plan.arena_bytes > 0
    rp, toks = Replay(drv), list(range(1, 130))
    a = run_cuts(rp, "a", toks, [])
    assert np.median(error(run_cuts(rp, "b", toks, [60, 100, 128]), a)) < 0.03


def test_bytes_of_pages_and_slots():
    from pie_b200.driver import memory_planner as mp
    from pie_b200.driver.kv_cache import KVCache
    from pie_b200.driver.recurrent import RecurrentStateCache
    cfg = ModelConfig.from_hf(nm.CONFIGS["mixed"])
    assert mp.kv_bytes_per_page(cfg, 16) == 2 * 16 * (2 * 64 * (2 + 2 + 2 + 4 + 4) + 64)
    kv = KVCache(0, 4, 1, 16, 64, torch.float32, "cpu", layer_shapes=cfg.kv_page_shapes(16))
    assert kv.data[2].shape == (5, 16, 64) and kv.data[4].shape == (5, 2, 4, 16, 64)
    assert kv.page_bytes_all_layers == 2 * mp.kv_bytes_per_page(cfg, 16)
    rs = RecurrentStateCache(cfg, 3, "cpu")
    assert rs.bytes_per_slot == 4 * (2 * 16 * 24 + 2 * 16 + 4 + 3 * 40 * 16 + 3 * 40 + 4) and set(rs.linear_at) == {0, 5}
    rs.linear_state[1] = torch.arange(rs.linear_state.shape[1])
    rs.copy_slot(1, 2)
    assert torch.equal(rs.linear_state[1], rs.linear_state[2]) and not rs.linear_state[0].any()
    assert mp.arena_bytes(cfg, 1024, 8) > 1024 * 96 * 16
    assert RecurrentStateCache(ModelConfig.from_hf(nm.CONFIGS["stateless"]), 2, "cpu").linear_at == {}
