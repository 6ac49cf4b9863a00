"""The Mananex design against the plain implementation in ``mananex_oracle``: whole prompts, decoding, portions, mixed
batches, used pages and slots, long decoding, and greedy generation through the engine's own scheduler."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import mananex_case as case
import mananex_oracle as oracle
import nisasun_case as nc
from legion_b200.config import DenseSpec, LayerSpec, MoeSpec, PRESETS, Hgrn2Spec, ModelConfig
from legion_b200.engine.lm import EngineConfig, LmEngine, build_engine
from legion_b200.engine.memory_plan import workspace_reserve
from legion_b200.engine.replay import TraceReplay, replay_engine
from legion_b200.engine.types import GenerateRequest, SamplingParams
from legion_b200.hw.gpu import model_bytes_per_step
from legion_b200.kv.blocks import OutOfBlocks
from legion_b200.loaders.model import load_model
from legion_b200.models.decoder import Decoder
from legion_b200.models.weights import weight_shapes

gpu = pytest.mark.gpu
WHERE = [pytest.param("cpu", "float32", id="cpu"), pytest.param("cuda:0", "float32", id="gpu-f32", marks=gpu),
         pytest.param("cuda:0", "bfloat16", id="gpu-bf16", marks=gpu)]


def check(got, want, dtype, what=""):
    e = nc.errors(got, want)
    if dtype == "float32":
        assert e.max() < 1e-4, (what, float(e.max()), int(e.argmax()))
    else:                                      # bf16 rounding
        assert e.max() < 0.1 and e.median() < 0.03, (what, float(e.median()), float(e.max()), int(e.argmax()))


def all_chosen(cfg):
    """The same with every expert chosen: a choice that rounding flips would change all later tokens (bf16 comparisons of
    whole models; which experts are chosen is tested alone)."""
    cfg = copy.deepcopy(cfg)
    for layer in cfg["layers"]:
        if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
            layer["mlp"]["router"]["top"] = layer["mlp"]["router"]["experts"]
    return cfg


class Models:
    def __init__(self, root):
        self.root, self.made, self.want = root, {}, {}

    def get(self, name, dtype="float32"):
        """(config, weights, directory); bf16 comparisons take the variant without close choices."""
        key = (name, dtype == "bfloat16")
        if key not in self.made:
            cfg = all_chosen(case.CASES[name]) if key[1] else case.CASES[name]
            w = case.make_weights(cfg, seed=list(case.CASES).index(name))
            self.made[key] = (cfg, w, nc.write_checkpoint(self.root / f"{name}{int(key[1])}", cfg, w))
        return self.made[key]

    def expected(self, name, dtype, n, seed):
        key = (name, dtype == "bfloat16", n, seed)
        if key not in self.want:
            cfg, w, _ = self.get(name, dtype)
            toks = nc.tokens(cfg, n, seed)
            self.want[key] = (toks, oracle.forward(cfg, w, toks))
        return self.want[key]

    def replay(self, name, device, dtype, max_tokens):
        return TraceReplay(replay_engine(self.get(name, dtype)[2], getattr(torch, dtype), max_tokens, device))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    return Models(tmp_path_factory.mktemp("mananex"))


def test_registry_and_config_round_trip():
    for name in ("tiny-mananex", "mananex-4b", "mananex-13b"):
        c = PRESETS[name]()
        assert ModelConfig.from_dict(json.loads(c.to_json())) == c
        assert len(c.layers) == c.n_layer == len(c.layer_kinds)
    c = PRESETS["tiny-mananex"]()
    assert c.kv_layers() == [0, 1, 2, 3] == c.recurrent_layers() and c.kv_dims(0) == (2, 32, 48)
    assert isinstance(c.recurrent_spec(2), Hgrn2Spec) and c.state_floats(2) == 2 * 64 * 40 and c.merged_output(1)
    s = weight_shapes(c)
    assert "output" not in s and "l0.ffn_norm" not in s and "l2.moe.router" not in s
    assert s["l3.dwa"] == (5,) and s["l2.rg_b"] == (144,) and s["l0.rg_b"] == (288,) and s["l0.mlp.gate_up_b"] == (400,)
    assert s["l1.moe.router_bias"] == (10,) and s["l1.mix.o"] == (144, 4 * 24 + 5 * 32)
    col = c.mix_columns(3)                       # every part of the stacked projection starts on a 16-byte boundary
    assert list(col) == ["q", "k", "v", "g", "rq", "rf", "rv", "rg1", "rg2", "end"]
    assert all(v % 8 == 0 for v in col.values()) and col["g"] == 3 * 40 + 40 + 32 and col["rq"] == col["g"] + 8
    assert model_bytes_per_step(c, 4, 100)["total_bytes"] > 0
    assert c.stream_rows() == 8 and PRESETS["tiny-gurozen"]().stream_rows() == 0
    reserve = [workspace_reserve(144, 512, 1000, 4, 0, 0, 0, n) for n in (0, c.stream_rows())]
    assert reserve[1] - reserve[0] == 1000 * 144 * 4 * 8
    with pytest.raises(ValueError, match="parallel sublayers"):
        ModelConfig(layers=[LayerSpec(Hgrn2Spec(1, 8, 8), DenseSpec(8, bias=True))])


def test_fresh_checkouts_compile_the_kernels_of_the_model_only():
    from legion_b200 import build_ext
    mine = build_ext.kernels_of(PRESETS["tiny-mananex"]())
    assert all((build_ext.CSRC / (k + ".cu")).exists() for k in mine)
    assert {"forget_scan", "forget_scan_sm100", "depth_step", "qkv_conv", "hyper", "moe", "attn_general"} <= mine
    assert not mine & {"latent_attn", "diag_scan", "resid_step", "linear_scan", "gdn", "channel_delta"}
    others = set().union(*(build_ext.kernels_of(PRESETS[n]()) for n in ("tiny-nisasun", "tiny-gurozen", "tiny-pemezen")))
    assert not others & {"forget_scan", "depth_step"}


@pytest.mark.parametrize("name", list(case.CASES))
def test_loader_maps_every_tensor(models, name):
    cfg, w, path = models.get(name)
    mc, lw, _, _ = load_model(path)
    shapes = weight_shapes(mc)
    assert set(shapes) == set(lw) and all(tuple(lw[k].shape) == tuple(v) for k, v in shapes.items())
    pad = 0
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}"
        spec, col, rows = mc.layers[i], mc.mix_columns(i), lw[f"{p}.mix.in"]
        parts = {"q": "mix.left.q", "k": "mix.left.k", "v": "mix.left.v", "g": "mix.left.g", "rq": "mix.right.q", "rf": "mix.right.f",
                 "rv": "mix.right.v", "rg1": "rg1", "rg2": "rg2"}
        for part, n in parts.items():
            if part != "rg2" or f is not None:
                t = w[f"{p}.{n}"].float()
                assert torch.equal(rows[col[part]:col[part] + t.shape[0]], t)
        pad += (col["end"] - sum(w[f"{p}.{n}"].shape[0] for n in parts.values() if f"{p}.{n}" in w)) * cfg["width"]
        a, s, nl = m["left"], spec.mixer, m["left"]["heads"] * m["left"]["vdim"]
        assert torch.equal(lw[f"{p}.mix.o"][:, :nl], w[f"{p}.mix.left.o"].float())
        assert torch.equal(lw[f"{p}.mix.o"][:, nl:], w[f"{p}.mix.right.o"].float())
        assert (s.left.window, s.left.keep_first, s.left.scale, s.left.rot.dims) == (
            a["mask"]["size"], a["mask"]["keep_first"], a["scale"], a["rot"]["dims"])
        assert (s.left_scale, s.right_scale, s.right.heads) == (m["left_scale"], m["right_scale"], m["right"]["heads"])
        assert f is None or isinstance(spec.mlp, DenseSpec if f["kind"] == "dense" else MoeSpec)
    assert sum(t.numel() for t in lw.values()) == sum(t.numel() for t in w.values()) + pad


def test_loader_without_optional_parts(tmp_path):
    """No rotation, no window, no feed-forward part."""
    cfg = case.config(64, 50, [case.layer(case.left(2, 1, 16, 16, 8, 2, 0), case.right(2, 16, 16), None)])
    w = case.make_weights(cfg, 3)
    plain = copy.deepcopy(cfg)
    del plain["layers"][0]["mixer"]["left"]["rot"], plain["layers"][0]["mixer"]["left"]["mask"], plain["layers"][0]["mlp"]
    path = nc.write_checkpoint(tmp_path, plain, w)
    cfg["layers"][0]["mixer"]["left"]["mask"]["size"] = 100
    toks = nc.tokens(cfg, 20, 1)
    r = TraceReplay(replay_engine(path, torch.float32, 64, "cpu"))
    check(nc.run_schedule(r, {"a": toks}, [[("a", 12)], [("a", 8)]])["a"], oracle.forward(cfg, w, toks), "float32")


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(case.CASES))
def test_whole_prompt_layer_by_layer(models, name, device, dtype):
    cfg, w, path = models.get(name, dtype)
    toks = nc.tokens(cfg, 70, 1)
    layers = []
    want = oracle.forward(cfg, w, toks, layers_out=layers)
    eng = replay_engine(path, getattr(torch, dtype), 128, device)
    assert eng.mcfg.n_layer == len(layers)
    s = eng.open_sequence("a")
    s.tokens, s.phase = list(toks), "prefill"
    s.table.ensure(eng.pool, len(toks))
    b = eng.build_batch_explicit([(s, 0, toks)], all_logits=True)
    b.capture_layers = list(range(len(layers)))
    out = eng.model.forward(b, eng.kv, eng.states)
    for i, x in enumerate(layers):
        check(out.captures[i].cpu(), x, dtype, f"layer {i}")
    check(out.logits.cpu(), want, dtype)


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(case.CASES))
def test_decoding_and_portions_equal_the_whole_prompt(models, name, device, dtype):
    toks, want = models.expected(name, dtype, 210, 2)
    n = len(toks)
    schedules = {
        "whole": [n],
        "decoded": [150] + [1] * (n - 150),
        "token by token": [1] * 72 + [n - 72],
        "twos": [2] * 20 + [60] + [2] * 10 + [n - 120],
        "odd": [63, 1, 65, 3, 64, n - 196],
        "page edges": [127, 2, 1, n - 130],
        "sevens": [7] * 30,
    }
    for what, cuts in schedules.items():
        assert sum(cuts) == n
        r = models.replay(name, device, dtype, n)
        got = nc.run_schedule(r, {"a": toks}, [[("a", c)] for c in cuts])["a"]
        check(got, want, dtype, f"{name}: {what}")
        assert r.engine.pool.used == 0 and len(r.engine._free_slots) == 4


@pytest.mark.parametrize("device,dtype", WHERE)
@pytest.mark.parametrize("name", list(case.CASES))
def test_unequal_batches_and_used_pages_and_slots(models, name, device, dtype):
    """Portions beside single tokens in one step; later sequences run in pages and slots that earlier ones left, in a
    pool that holds no more than the live ones need."""
    seqs, want = {}, {}
    for i, n in enumerate((130, 66, 1, 97, 64, 129, 40)):
        seqs[f"s{i}"], want[f"s{i}"] = models.expected(name, dtype, n, 10 + i)
    schedule = [[("s0", 50), ("s1", 1), ("s2", 1)],
                [("s0", 1), ("s1", 63), ("s3", 2)],
                [("s3", 90), ("s0", 78), ("s1", 1)],
                [("s1", 1), ("s0", 1), ("s3", 1), ("s4", 64)],          # s0, s1 and s4 end
                [("s3", 1), ("s5", 1)], [("s3", 1), ("s5", 1)],          # two decoded together
                [("s5", 120), ("s6", 3)], [("s5", 1), ("s6", 36), ("s3", 1)],
                [("s5", 1), ("s3", 1), ("s6", 1)]] + [[("s5", 1)]] * 5
    r = models.replay(name, device, dtype, 8 * 64)
    for turn in range(2):                                                # the second turn only sees used pages
        got = nc.run_schedule(r, seqs, schedule)
        for k in seqs:
            check(got[k], want[k], dtype, f"{name} {k} turn {turn}")
        assert r.engine.pool.used == 0
    with pytest.raises(OutOfBlocks):
        r.step([{"id": "big", "tokens": [0] * (8 * 64 + 1), "want": []}], [])


@pytest.mark.parametrize("device,dtype", WHERE)
def test_long_prompt_in_long_portions(models, device, dtype):
    toks, want = models.expected("wide", dtype, 700, 30)
    for cuts in ([700], [400, 1, 299], [513, 2, 2, 183]):
        r = models.replay("wide", device, dtype, 700)
        check(nc.run_schedule(r, {"a": toks}, [[("a", c)] for c in cuts])["a"], want, dtype, str(cuts))


@pytest.mark.parametrize("device,dtype", WHERE)
def test_long_decoding(models, device, dtype):
    toks, want = models.expected("mixed", dtype, 330, 40)
    r = models.replay("mixed", device, dtype, 330)
    got = nc.run_schedule(r, {"a": toks}, [[("a", 20)]] + [[("a", 1)]] * 310)["a"]
    check(got, want, dtype)
    if device != "cpu":
        assert r.engine._graphs.replays == 310                           # decode steps replay the captured graph


@pytest.mark.parametrize("device,dtype", WHERE[:2])
def test_greedy_generation_through_the_scheduler(models, device, dtype):
    """Concurrent requests of unequal length, prompts cut into chunks, a resumed prefix: the tokens of the plain
    implementation's greedy continuation."""
    cfg, w, path = models.get("mixed")
    mc, lw, tok, _ = load_model(path, device, getattr(torch, dtype))
    eng = LmEngine(Decoder(mc, lw, None, max_position=264), tok,
                   EngineConfig(ctx_size=256, max_seqs=3, block_size=16, prefill_chunk=24, max_batch_tokens=40,
                                prefix_cache=True, device=device))

    def greedy(prompt, n):
        t = list(prompt)
        for _ in range(n):
            t.append(int(oracle.forward(cfg, w, t)[-1].argmax()))
        return t[len(prompt):]
    prompts = [nc.tokens(cfg, n, 60 + n) for n in (5, 61, 33, 90)]
    want = [greedy(p, 6) for p in prompts]
    streams = [eng.generate(GenerateRequest(prompt_tokens=list(p), sampling=SamplingParams(
        temperature=0.0, max_tokens=6, ignore_eos=True))) for p in prompts]
    assert [s.collect().token_ids for s in streams] == want
    # a longer conversation over the cached prefix: pages and the states come back
    follow = prompts[3] + want[3] + nc.tokens(cfg, 9, 77)
    out = eng.generate_text(tokens=follow, temperature=0.0, max_tokens=4, ignore_eos=True)
    assert out.token_ids == greedy(follow, 4) and out.usage.cached_tokens > 0
    eng.shutdown()


def test_preempted_sequences_are_recomputed():
    c = PRESETS["tiny-mananex"]()
    prompts = [torch.randint(0, 256, (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (40, 33, 50)]

    def run(**kw):
        eng = build_engine(c, engine_cfg=EngineConfig(ctx_size=128, max_seqs=3, block_size=16, prefill_chunk=32,
                                                      prefix_cache=False, **kw))
        ss = [eng.generate(GenerateRequest(prompt_tokens=p, sampling=SamplingParams(temperature=0.0, max_tokens=40,
                                                                                   ignore_eos=True))) for p in prompts]
        out = [s.collect().token_ids for s in ss]
        n = eng.stats().kv_preemptions
        eng.shutdown()
        return out, n
    plain, _ = run()
    for extra in ({}, {"kv_swap_gib": 0.1}):
        tight, n = run(kv_admission="on-demand", kv_cache_tokens=12 * 16, **extra)
        assert tight == plain and n > 0


def test_speculation_and_ranks_are_refused():
    from legion_b200.models.weights import Shard
    c = PRESETS["tiny-mananex"]()
    with pytest.raises(ValueError, match="speculative"):
        build_engine(c, engine_cfg=EngineConfig(ctx_size=64, max_seqs=1, spec="ngram"), start=False)
    with pytest.raises(NotImplementedError):
        Shard(c, 0, 2)


@gpu
def test_sampled_generation_on_gpu():
    c = PRESETS["tiny-mananex"]()
    eng = build_engine(c, device="cuda:0", engine_cfg=EngineConfig(ctx_size=256, max_seqs=4, block_size=64))
    a = eng.generate_text(tokens=list(range(70)), temperature=0.8, top_k=20, max_tokens=12, seed=3, ignore_eos=True)
    b = eng.generate_text(tokens=list(range(70)), temperature=0.8, top_k=20, max_tokens=12, seed=3, ignore_eos=True)
    assert a.error is None and len(a.token_ids) == 12 and a.token_ids == b.token_ids
    eng.shutdown()


@gpu
@pytest.mark.parametrize("branches,lanes", [(3, 2), (0, 2), (0, 1)])
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_many_sequences_decode_together(models, dtype, branches, lanes, monkeypatch):
    """More decoded sequences than one routing tile holds, with sublayers on branches of the captured step, as two lanes of it,
    and in a row."""
    from legion_b200.ops import sm100
    monkeypatch.setitem(sm100.TUNE, "parallel_branches", branches)
    monkeypatch.setitem(sm100.TUNE, "decode_lanes", lanes)
    cfg, w, path = models.get("mixed", dtype)
    n = 70
    seqs = {f"q{i}": nc.tokens(cfg, 9 + i % 5, 200 + i) for i in range(n)}
    want = {k: oracle.forward(cfg, w, v) for k, v in list(seqs.items())[::9]}
    r = TraceReplay(replay_engine(path, getattr(torch, dtype), n * 64, "cuda:0", slots=n))
    first = [[(k, len(v) - 4) for k, v in seqs.items()]]
    got = nc.run_schedule(r, seqs, first + [[(k, 1) for k in seqs]] * 4)
    for k in want:
        check(got[k], want[k], dtype, k)


@gpu
@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_run_program(models, tmp_path, dtype):
    cfg, w, path = models.get("mixed", dtype)
    toks, want = models.expected("mixed", dtype, 66, 11)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[40:65], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[65:], "want": [0]}], "end": ["x"]}]
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=240)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (tmp_path / "1.f32").exists()
    for n, places in ((0, [0, 39]), (2, [65])):
        got = torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(len(places), -1)
        e = nc.errors(got, want[places])
        assert e.max() < (1e-4 if dtype == "float32" else 0.08), e
