"""Puzutar through the driver, the context manager and the engine, against the plain statement in puzutar_oracle.py:
whole prompts, token by token, portions, unequal batches, pages and state slots used again, window edges, long decoding,
greedy generation. Each runs on the CPU path (32-bit) and, on a GPU, on the kernels in 32-bit and in bf16."""
import json

import numpy as np
import pytest
import puzutar_models as pm
import puzutar_oracle as oracle
import torch

from pie_b200.driver.executor import TorchDriver
from pie_b200.inferlets import install_all
from pie_b200.models import loader
from pie_b200.models.config import ModelConfig
from pie_b200.runtime.engine import Engine, EngineConfig
from pie_b200.runtime.rs_cache import RsState
from pie_b200.runtime.tokenizer import ByteTokenizer
from pie_b200.runtime.trace import Replay

PATHS = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", "bfloat16"), id="cuda-bf16", marks=pytest.mark.gpu)]
# root mean square of the difference over the vocabulary, against the root mean square of the logits
LIMIT = {"float32": 2e-5, "bfloat16": 0.035}
_WANT: dict = {}


def want(name, n, seed=0):
    """Oracle logits of every position of the prompt (name, n, seed)."""
    key = (name, n, seed)
    if key not in _WANT:
        cfg = pm.CONFIGS[name]
        _WANT[key] = oracle.forward(cfg, pm.tensors(cfg), pm.prompt(cfg, n, seed)).numpy()
    return _WANT[key]


def error(got, ref):
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def make_driver(name, path, pages=40, slots=4, max_tokens=512, **kw):
    device, dtype = path
    cfg = ModelConfig.from_hf(pm.CONFIGS[name], name)
    t = pm.tensors(pm.CONFIGS[name])
    prog = loader.compile_program(cfg, list(t), dtype=dtype)
    w = loader.execute_program(prog, loader.TensorDictReader(t), device)
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
@pytest.mark.parametrize("name", list(pm.CONFIGS))
def test_whole_prompt_token_by_token_and_portions(name, path):
    n = 60 if path[0] == "cpu" else 200
    cfg = pm.CONFIGS[name]
    toks, ref = pm.prompt(cfg, n), want(name, n)
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
@pytest.mark.parametrize("name", ["shared", "odd", "heads"])
def test_unequal_batches_against_each_alone_with_pages_and_slots_reused(name, path):
    """Four live requests of unequal lengths in every step: portions beside single tokens, requests left out of steps,
    ended and replaced; the pool holds little more than the live tokens, so pages and slots change hands."""
    cfg = pm.CONFIGS[name]
    lens = [33, 50, 7, 64, 40, 18, 55, 1, 30]
    prompts = [pm.prompt(cfg, n, i) for i, n in enumerate(lens)]
    rng = np.random.default_rng(5)
    drv = make_driver(name, path, pages=16)
    rp, at, live, waiting = Replay(drv), {}, [], list(range(len(lens)))
    got = {i: [] for i in range(len(lens))}
    used = []
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        entries, end = [], []
        for i in [x for x in live if len(live) == 1 or rng.random() < 0.8] or live[:1]:
            k = min(int(rng.choice([1, 1, 2, 5, 17, 31])), lens[i] - at[i])
            entries.append((i, at[i], at[i] + k))
            at[i] += k
        order = rng.permutation(len(entries))
        entries = [entries[j] for j in order]
        end = [i for i, _, b in entries if b == lens[i]]
        rows = rp.step([entry(f"r{i}", prompts[i], a, b) for i, a, b in entries], [f"r{i}" for i in end])
        used.append(drv.kv.num_pages)
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
    n = 150 if path[0] == "cpu" else 330
    for name, page in (("shared", 16), ("odd", 32)):
        toks = pm.prompt(pm.CONFIGS[name], n)
        rp = Replay(make_driver(name, path, page_size=page), page)
        close(run_cuts(rp, "a", toks, list(range(20, n))), want(name, n), path[1])
        close(run_cuts(rp, "b", toks, [90]), want(name, n), path[1])


@pytest.mark.parametrize("path", PATHS)
def test_padded_buckets_do_not_touch_the_state(path):
    """Three single-token requests run in a bucket of four; a fourth request left out meanwhile goes on unharmed."""
    cfg = pm.CONFIGS["shared"]
    prompts = [pm.prompt(cfg, 24, i) for i in range(4)]
    rp = Replay(make_driver("shared", path))
    rows = [[r] for r in np.split(rp.step([entry(f"r{i}", prompts[i], 0, 9) for i in range(4)]), 4)]
    for s in range(9, 24):
        ids = [0, 1, 2] if s < 16 else [0, 1, 2, 3]
        spans = [(i, s if i < 3 else s - 7) for i in ids]
        out = rp.step([entry(f"r{i}", prompts[i], a, a + 1) for i, a in spans])
        for (i, _), r in zip(spans, out):
            rows[i].append(r[None])
    for i in range(4):
        got = np.concatenate(rows[i])
        close(got, want("shared", 24, i)[:len(got)], path[1])


def sensitivity(kind):
    """Relative change of the logits when the plain statement itself is wrong in one way."""
    cfg = json.loads(json.dumps(pm.CONFIGS["shared"]))
    t, toks = pm.tensors(cfg), pm.prompt(cfg, 120)
    good = oracle.forward(cfg, t, toks)
    save = {}

    def swap(name, fn):
        save[name] = getattr(oracle, name)
        setattr(oracle, name, fn)
    if kind in ("window+1", "window-1"):
        for spec in cfg["layers"]:
            spec["mixer"]["mask"]["size"] += 1 if kind == "window+1" else -1
    elif kind == "shift lost at 60":
        swap("token_shift", lambda h, mix: h + (torch.cat([torch.zeros_like(h[:1]), h[:-1]]).index_fill(0, torch.tensor([60]), 0.0) - h) * mix)
    elif kind == "one group":
        swap("grouped_norm", lambda x, w, g, eps: oracle.rms(x, eps) * w)
    elif kind == "own key":
        for spec in cfg["layers"]:
            spec["mixer"].pop("kv_from", None)
        t = dict(t)
        for i in (1, 3):
            t[f"l{i}.mix.dkv"], t[f"l{i}.mix.dkv.norm"] = t["l0.mix.dkv"], t["l0.mix.dkv.norm"]
    elif kind == "side without the token":
        swap("token_side", lambda x, e, gate, proj, w, eps: x + oracle.rms(oracle.gelu_tanh(x @ gate.t()) @ proj.t(), eps) * w)
    try:
        bad = oracle.forward(cfg, t, toks)
    finally:
        for k, v in save.items():
            setattr(oracle, k, v)
    return error(bad.numpy(), good.numpy())[60:].max()


@pytest.mark.parametrize("kind", ["window+1", "window-1", "shift lost at 60", "one group", "own key", "side without the token"])
def test_the_models_show_mistakes(kind):
    """A mistake planted in the plain statement moves the logits well past the tolerance of the bf16 comparisons."""
    assert sensitivity(kind) > 3 * LIMIT["bfloat16"]


# ------------------------------------------------------------------ configuration, loading, engine
def test_configuration_and_registry(tmp_path):
    cfg = ModelConfig.from_hf(pm.CONFIGS["odd"])
    assert cfg.model_type == "puzutar" and cfg.ff_sizes == [70, 0, 21] and cfg.latent_cache_layers == [0, 1]
    assert cfg.latent_cache_index == {0: 0, 1: 1, 2: 0} and cfg.plan_window_left == 199 and cfg.recurrent_layers == [0, 1, 2]
    assert cfg.kv_elems_per_page(1) == 2 * cfg.latent_row
    bad = json.loads(json.dumps(pm.CONFIGS["shared"]))
    bad["layers"][1]["mixer"]["kv_rank"] = 24
    with pytest.raises(ValueError, match="kv_from"):
        ModelConfig.from_hf(bad)
    bad = json.loads(json.dumps(pm.CONFIGS["shared"]))
    bad["layers"][0]["mixer"]["kv_from"] = 2
    with pytest.raises(ValueError, match="kv_from"):
        ModelConfig.from_hf(bad)
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["norm"].update(groups=7)):
        bad = json.loads(json.dumps(pm.CONFIGS["shared"]))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)


def test_checkpoint_round_trip_and_type_check(tmp_path):
    cfg_d = pm.CONFIGS["odd"]
    t = pm.tensors(cfg_d)
    cfg, w = loader.load_checkpoint(pm.write_checkpoint(tmp_path / "a", cfg_d, t), "cpu", dtype="bfloat16")
    loader.export_hf_checkpoint(cfg, w, tmp_path / "b")
    from safetensors.torch import load_file
    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    assert ModelConfig.from_path(tmp_path / "b").latent == cfg.latent
    t["l1.mix.uv"] = t["l1.mix.uv"][:-1]
    with pytest.raises(loader.LoaderTypeError, match="l1.mix.uv"):
        loader.load_checkpoint(pm.write_checkpoint(tmp_path / "c", cfg_d, t), "cpu")


def oracle_greedy(name, toks, n):
    cfg, toks = pm.CONFIGS[name], list(toks)
    k = len(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, pm.tensors(cfg), toks)[-1].argmax()))
    return toks[k:]


@pytest.mark.parametrize("path", PATHS[:2])
def test_greedy_generation_through_the_engine(path):
    """Entry point, scheduler, chunked prefill (the prompt exceeds a pass), more contexts than state slots; fork and a lost
    state that is rebuilt from the lineage."""
    name = "shared"
    drv = make_driver(name, path, pages=64, slots=8, max_tokens=48)
    drv.rs.num_slots = 3
    e = Engine(EngineConfig())
    e.add_model("m", drv, tokenizer=ByteTokenizer(pm.CONFIGS[name]["vocab"]))
    install_all(e)
    try:
        prompts = [pm.prompt(pm.CONFIGS[name], n, i) for i, n in enumerate((70, 9, 30, 50))]
        pids = [e.launch("text-completion", {"prompt_tokens": p, "max_tokens": 6, "temperature": 0.0, "stop_tokens": []})
                for p in prompts]
        outs = [json.loads(e.wait(p, 300))["tokens"] for p in pids]
        assert outs == [oracle_greedy(name, p, 6) for p in prompts]
        from pie_b200.sdk import Context, Model, Sampler

        async def prog(args):
            ctx = Context(Model.load("m"))
            ctx.append(prompts[2])
            first = await ctx.generate(Sampler.argmax(), max_tokens=3).stop([]).collect_tokens()
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
