"""Vulanex through the driver, the context manager and the engine, against the plain statement in vulanex_oracle.py: whole
prompts, token by token, portions, unequal batches, pages and state slots used again, edges of windows and of pooled blocks, first
tokens, long decoding, greedy generation. Each runs on the CPU path (32-bit) and, on a GPU, on the kernels in 32-bit and in
bf16."""
import json

import numpy as np
import pytest
import torch
import vulanex_models as vm
import vulanex_oracle as oracle

from pie_b200.driver.executor import TorchDriver
from pie_b200.inferlets import install_all
from pie_b200.models import loader
from pie_b200.models.block_spec import EVERYTHING, DeltaRuleSpec, ParallelSpec, PlainAttentionSpec
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
        _TENSORS[name] = vm.tensors(vm.CONFIGS[name])
    return _TENSORS[name]


def want(name, n, seed=0):
    """Oracle logits of every position of the prompt (name, n, seed)."""
    if (name, n, seed) not in _WANT:
        cfg = vm.CONFIGS[name]
        _WANT[name, n, seed] = oracle.forward(cfg, tensors(name), vm.prompt(cfg, n, seed)).numpy()
    return _WANT[name, n, seed]


def error(got, ref):
    d = got - ref
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((ref ** 2).mean())


def make_driver(name, path, pages=40, slots=4, max_tokens=512, **kw):
    device, dtype = path
    cfg, t = ModelConfig.from_hf(vm.public(vm.CONFIGS[name])), tensors(name)
    reader = loader.TensorDictReader(t)
    loader.complete_blocks(cfg, reader)
    w = loader.execute_program(loader.compile_program(cfg, list(t), dtype=dtype), reader, device)
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
@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_whole_prompt_token_by_token_and_portions(name, path):
    n = 56 if path[0] == "cpu" else 200
    toks, ref = vm.prompt(vm.CONFIGS[name], n), want(name, n)
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
    ended and replaced; the pool holds little more than the live tokens, so pages, means and slots change hands."""
    cfg = vm.CONFIGS[name]
    lens = [33, 50, 7, 64, 40, 18, 55, 1, 30]
    if path[0] != "cpu":
        lens[3] = 150                                   # several key blocks and pieces beside short portions
    prompts = [vm.prompt(cfg, n, i) for i, n in enumerate(lens)]
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
        toks = vm.prompt(vm.CONFIGS[name], n)
        rp = Replay(make_driver(name, path, page_size=page), page)
        close(run_cuts(rp, "a", toks, list(range(20, n))), want(name, n), path[1])
        close(run_cuts(rp, "b", toks, [90]), want(name, n), path[1])


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_prompts_of_many_rows_in_one_batch(name):
    """Batches past the rows from which norms and convolutions run in two launches."""
    cfg, lens = vm.CONFIGS[name], [300, 2, 320, 17]
    rp = Replay(make_driver(name, ("cuda", "bfloat16"), pages=60, max_tokens=1024))
    prompts = [vm.prompt(cfg, n, i) for i, n in enumerate(lens)]
    rows = rp.step([entry(f"r{i}", t, 0, len(t)) for i, t in enumerate(prompts)], [f"r{i}" for i in range(4)])
    for i, got in enumerate(np.split(rows, np.cumsum(lens)[:-1])):
        close(got, want(name, lens[i], i), "bfloat16")


@pytest.mark.parametrize("path", PATHS)
def test_padded_buckets_do_not_touch_the_state(path):
    """Three single-token requests run in a bucket of four; a fourth request left out meanwhile goes on unharmed."""
    cfg = vm.CONFIGS["mixed"]
    prompts = [vm.prompt(cfg, 24, i) for i in range(4)]
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


def swapped(kind, cfg, t):
    """Plant one mistake in the plain statement (returns {name: replacement}), its configuration or its tensors."""
    o = {k: getattr(oracle, k) for k in dir(oracle)}
    masks = [s["mixer"]["left"]["mask"] for s in cfg["layers"] if "left" in s["mixer"]]
    pair = cfg["embedding"]["bigram"]
    if kind in ("window+1", "window-1"):
        for m in masks:
            m["size"] += 1 if kind == "window+1" else -1
    elif kind == "longer blocks":
        for m in masks:
            m["pool"] += 1
    elif kind == "pair factors swapped":
        pair["mul_prev"], pair["mul_cur"] = pair["mul_cur"], pair["mul_prev"]
    elif kind == "frequencies unscaled":
        for s in cfg["layers"]:
            s["mixer"].get("left", {}).get("rot", {}).pop("scaling", None)
    elif kind == "factor by other positions":
        for s in cfg["layers"]:
            if "q_temp" in s["mixer"]:
                s["mixer"]["q_temp"]["every"] *= 2
    elif kind == "logits unscaled":
        cfg["logit_scale"] = 1.0
    elif kind in ("no norm offsets", "no sublayer gain"):
        for k in t:
            if k.endswith(("norm1.b", "norm2.b") if kind == "no norm offsets" else (".left.out", ".right.out")):
                t[k] = torch.zeros_like(t[k]) if kind == "no norm offsets" else torch.ones_like(t[k])
    lost = lambda f, x, *rest: torch.cat([f(x[:60], *rest), f(x[60:], *rest)])
    return {
        "no sink": {"weights_with_sink": lambda s, see, sink: torch.softmax(s.masked_fill(~see, float("-inf")), -1)},
        "block a token early": {"seen_blocks": lambda t, size, pool: o["seen_blocks"](t, size - 1, pool)},
        "block a token late": {"seen_blocks": lambda t, size, pool: o["seen_blocks"](t, size + 1, pool)},
        "no blocks": {"seen_blocks": lambda t, size, pool: torch.zeros_like(o["seen_blocks"](t, size, pool))},
        "sums for means": {"block_means": lambda x, pool: o["block_means"](x, pool) * pool},
        "cos and sin unscaled": {"stretched_frequencies": lambda rot: (o["stretched_frequencies"](rot)[0], 1.0)},
        "no first-token row": {"embedding": lambda tokens, embed, bigram, mul_prev, mul_cur, buckets: o["embedding"](
            tokens, embed, torch.cat([bigram[:-1], 0 * bigram[-1:]]), mul_prev, mul_cur, buckets)},
        "token before lost at 60": {"embedding": lambda tokens, *a, **k: torch.cat([o["embedding"](tokens[:60], *a, **k),
                                                                                  o["embedding"](tokens[60:], *a, **k)])},
        "history lost at 60": {"input_convolution": lambda h, w: lost(o["input_convolution"], h, w)},
        "convolution alone": {"input_convolution": lambda h, w: o["input_convolution"](h, w) - h},
        "taps reversed": {"input_convolution": lambda h, w: o["input_convolution"](h, w.flip(1))},
        "state lost at 60": {"delta_rule": lambda r, k, v, w, a: (torch.cat([o["delta_rule"](*(x[s] for x in (r, k, v, w, a)))[0]
                                                                           for s in (slice(0, 60), slice(60, None))]), None)},
        "keys as they are": {"unit": lambda k: k},
        "nothing removed": {"removal_rates": lambda h, w: 0 * o["removal_rates"](h, w)},
        "other decays": {"decays": lambda h, w: o["decays"](h, w) ** 1.5},
        "no query factor": {"query_factor": lambda p, coef, every: torch.ones_like(p)},
        "sum for mean norm": {"layer_norm": lambda x, w, b, eps: o["rms"](x, eps) * w + b},
        "other activation": {"gelu_tanh": lambda z: z * o["sigmoid"](z)},
    }.get(kind, {})


KINDS = ["window+1", "window-1", "longer blocks", "no sink", "block a token early", "block a token late", "no blocks", "sums for means",
         "frequencies unscaled", "cos and sin unscaled", "pair factors swapped", "no first-token row", "token before lost at 60",
         "history lost at 60", "convolution alone", "taps reversed", "state lost at 60", "keys as they are", "nothing removed",
         "other decays", "no query factor", "factor by other positions", "sum for mean norm", "other activation", "logits unscaled",
         "no norm offsets", "no sublayer gain"]


# one mean more or less among many keys, a factor of nearly the same size: the 32-bit comparisons show it, and those of the ops
# alone in bf16
SUBTLE = {"window+1", "window-1", "block a token early", "block a token late", "factor by other positions"}


@pytest.mark.parametrize("kind", KINDS)
def test_the_models_show_mistakes(kind, monkeypatch):
    """A mistake planted in the plain statement moves the logits well past the tolerance of the comparisons."""
    cfg, t, toks = json.loads(json.dumps(vm.CONFIGS["mixed"])), dict(tensors("mixed")), vm.prompt(vm.CONFIGS["mixed"], 110)
    good = want("mixed", 110)
    for name, fn in swapped(kind, cfg, t).items():
        monkeypatch.setattr(oracle, name, fn)
    e = error(oracle.forward(cfg, t, toks).numpy(), good)
    limit = 100 * LIMIT["float32"] if kind in SUBTLE else 2 * LIMIT["bfloat16"]
    assert not (e[0] if kind == "no first-token row" else e[60:].max()) <= limit            # (a state may also grow without bound)


# ------------------------------------------------------------------ configuration, loading, engine
def test_configuration_and_registry():
    cfg = ModelConfig.from_hf(vm.public(vm.CONFIGS["mixed"]))
    assert cfg.model_type == "vulanex" and cfg.stream32 and cfg.layer_norm and cfg.conv_taps == 3 and cfg.logit_scale == 0.7
    assert [type(b.mixer) for b in cfg.blocks] == [ParallelSpec, PlainAttentionSpec, ParallelSpec, PlainAttentionSpec]
    assert isinstance(cfg.blocks[0].recurrent, DeltaRuleSpec) and cfg.blocks[1].recurrent is None and cfg.blocks[0].mixer.out_norms
    assert cfg.kv_layers == [(2, 64, 2, 6), (2, 64, 1, 0), (4, 64, 2, 12), (1, 64, 1, 0)] and cfg.plan_window_left == -1
    a = cfg.blocks[3].attention
    assert a.shared_kv and a.window == EVERYTHING and a.q_temp == (0.4, 7) and a.planes == 1 and not a.sink and a.rot is None
    assert cfg.blocks[0].ff.act == "gelu_tanh" and cfg.token_pairs.buckets == 61
    left = lambda c: c["layers"][0]["mixer"]["left"]
    for change in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][1]["mixer"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"].update(vdim=16),
                   lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), lambda c: left(c)["mask"].update(size=0),
                   lambda c: left(c)["mask"].update(pool=0), lambda c: left(c)["rot"].update(dims=42), lambda c: left(c)["rot"].update(dims=5),
                   lambda c: c["canon"].update(taps=0), lambda c: c["embedding"]["bigram"].update(buckets=0)):
        bad = json.loads(json.dumps(vm.public(vm.CONFIGS["mixed"])))
        change(bad)
        with pytest.raises(ValueError):
            ModelConfig.from_hf(bad)
    assert preset("vulanex-8b", num_hidden_layers=3).num_hidden_layers == 3


@pytest.mark.parametrize("name", list(vm.CONFIGS))
def test_checkpoint_round_trip_and_type_check(tmp_path, name):
    cfg_d, t = vm.CONFIGS[name], dict(tensors(name))
    cfg, w = loader.load_checkpoint(vm.write_checkpoint(tmp_path / "a", cfg_d, t), "cpu", dtype="bfloat16")
    loader.export_hf_checkpoint(cfg, w, tmp_path / "b")
    from safetensors.torch import load_file
    back = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(back) == set(t) and all(torch.equal(back[k], t[k]) for k in t)
    again, _ = loader.load_checkpoint(tmp_path / "b", "cpu")
    assert again.blocks == cfg.blocks and again.logit_scale == cfg.logit_scale and again.token_pairs == cfg.token_pairs
    for key in ("bigram", next(k for k in t if k.endswith(".canon1"))):
        bad = dict(t)
        bad[key] = torch.cat([t[key], t[key][:, :1]], 1) if key != "bigram" else t[key][:-1]
        with pytest.raises(loader.LoaderTypeError, match=key):
            loader.load_checkpoint(vm.write_checkpoint(tmp_path / "c", cfg_d, bad), "cpu")


def oracle_greedy(name, toks, n):
    toks, k = list(toks), len(toks)
    for _ in range(n):
        toks.append(int(oracle.forward(vm.CONFIGS[name], tensors(name), toks)[-1].argmax()))
    return toks[k:]


@pytest.mark.parametrize("path", PATHS[:2])
def test_greedy_generation_through_the_engine(path):
    """Entry point, scheduler, chunked prefill (the prompt exceeds a pass), more contexts than state slots; fork and a lost
    state that is rebuilt from the lineage."""
    name = "mixed"
    drv = make_driver(name, path, pages=64, slots=8, max_tokens=48)
    drv.rs.num_slots = 3
    e = Engine(EngineConfig())
    e.add_model("m", drv, tokenizer=ByteTokenizer(vm.CONFIGS[name]["vocab"]))
    install_all(e)
    try:
        prompts = [vm.prompt(vm.CONFIGS[name], n, i) for i, n in enumerate((70, 9, 30, 50))]
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
    cfg = preset("tiny-vulanex")
    drv = TorchDriver(cfg, "cuda", num_pages=0, max_requests=8, max_tokens=512, gpu_mem_utilization=0.3)
    assert drv.rs.num_slots == 16 and drv.kv.num_pages >= 64 and drv.memory_plan.arena_bytes > 0
    rp, toks = Replay(drv), list(range(1, 130))
    a = run_cuts(rp, "a", toks, [])
    assert np.median(error(run_cuts(rp, "b", toks, [60, 100, 128]), a)) < 0.03


def test_bytes_of_pages_and_slots():
    from pie_b200.driver import memory_planner as mp
    from pie_b200.driver.kv_cache import KVCache
    from pie_b200.driver.recurrent import RecurrentStateCache
    from pie_b200.driver.schema import CopyDir, CopyRequest
    cfg = ModelConfig.from_hf(vm.public(vm.CONFIGS["mixed"]))
    # rows of two planes or one; three (two) means per page of the layers with blocks of six (twelve)
    elems = 64 * (2 * 2 * (16 + 3) + 2 * 16 + 2 * 4 * (16 + 2) + 16)
    assert mp.kv_bytes_per_page(cfg, 16) == 2 * elems
    kv = KVCache(0, 4, 1, 16, 64, torch.float32, "cpu", swap_pages=2, layer_shapes=cfg.kv_page_shapes(16))
    assert kv.data[1].shape == (5, 1, 2, 16, 64) and kv.data.means[0].shape == (5, 2, 2, 3, 64) and kv.data.means[1] is None
    assert kv.data.means[2].shape == (5, 2, 4, 2, 64) and kv.page_bytes_all_layers == 4 * elems
    kv.data.means[2][1] = 3.0
    kv.copy(CopyRequest(CopyDir.D2D, [1], [2]))
    kv.copy(CopyRequest(CopyDir.D2H, [1], [0]))
    kv.copy(CopyRequest(CopyDir.H2D, [0], [3]))
    assert (kv.data.means[2][2] == 3).all() and (kv.data.means[2][3] == 3).all() and not kv.data.means[2][0].any()
    rs = RecurrentStateCache(cfg, 3, "cpu")
    assert set(rs.linear_at) == {0, 2} and rs.bytes_per_slot == 4 * (2 * 24 * 24 + 3 * 40 * 40 + 8 * 2 * 96 + 4)
    assert sorted(rs.carried["history_at"]) == [(li, h) for li in range(4) for h in ("1", "2")]
    rs.linear_state[1] = torch.arange(rs.linear_state.shape[1])
    rs.copy_slot(1, 2)
    assert torch.equal(rs.linear_state[1], rs.linear_state[2]) and not rs.linear_state[0].any()
    assert mp.arena_bytes(cfg, 1024, 8) > 1024 * 96 * 16
    bare = RecurrentStateCache(ModelConfig.from_hf(vm.public(vm.CONFIGS["tall"])), 2, "cpu")
    assert bare.carried["history_at"] == {} and bare.linear_state.shape[1] == 136 * 136 + 2 * 30 * 30 + 4
