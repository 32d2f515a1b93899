"""Zedirax end to end: checkpoint -> loader -> pages and state slots -> engine step, against the plain reference of ``zedirax_oracle``
(float64).  Every test runs on the CPU references of the ops and, on a GPU box, on the kernels."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from . import zedirax_cases as C
from . import zedirax_oracle as O
from . import layerspec_cases as L
from gemm_b200.models import loader
from gemm_b200.models.config import ModelConfig, get_config
from gemm_b200.serve.engine import Engine, SamplingParams
from gemm_b200.serve.llm import LLM
from gemm_b200.serve.replay import Replay

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
FORMATS = ["f32", "bf16"]
TOL, RMS = {"f32": 3e-4, "bf16": 8e-2}, {"f32": 3e-5, "bf16": 3e-2}      # of the worst position, and over all
PAGE = 64
_models, _logits = {}, {}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    return tmp_path_factory.mktemp("zedirax")


def get_model(name):
    if name not in _models:
        _models[name] = C.make_model(name)
    return _models[name]


def want(name, n, seed):
    """Tokens and the reference's logits of a sequence (computed once)."""
    key = (name, n, seed)
    if key not in _logits:
        toks = L.tokens(get_model(name), n, seed)
        _logits[key] = (toks, O.forward(get_model(name), toks))
    return _logits[key]


def weights(folder, name, fmt, device):
    path = os.path.join(str(folder), name)
    if not os.path.exists(path):
        C.save_model(get_model(name), path)
    return loader.load_safetensors(path, fmt, device)


def make_llm(folder, name, fmt, device, pages=12, slots=4, page=PAGE, **kw):
    return LLM(weights(folder, name, fmt, device), None, max_running=slots, num_pages=pages, page_size=page, **kw)


def assert_close(got, ref, fmt, what=""):
    e = L.err(got, ref)
    assert bool(torch.isfinite(e).all()), what
    assert e.max() < TOL[fmt] and e.pow(2).mean().sqrt() < RMS[fmt], (what, int(e.argmax()), float(e.max()), float(e.pow(2).mean().sqrt()))


def check_ok(device):
    if device == "cuda":
        from gemm_b200 import _native
        _native.assert_status_ok()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_whole_prompt(folder, name, fmt, device):
    toks, ref = want(name, 203, 0)
    got = L.replay_one(Replay(make_llm(folder, name, fmt, device)), toks, [203])
    check_ok(device)
    assert_close(got, ref, fmt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
@pytest.mark.parametrize("sizes", [[2], [64], [65, 1, 63, 2, 3], [130, 7]])
def test_portions(folder, sizes, fmt, device):
    for name in ("mixed", "wide"):
        toks, ref = want(name, 203, 0)
        got = L.replay_one(Replay(make_llm(folder, name, fmt, device)), toks, L.cuts(203, sizes))
        check_ok(device)
        assert_close(got, ref, fmt, name)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
@pytest.mark.parametrize("name", sorted(C.CASES))
def test_token_by_token(folder, name, fmt, device):
    """Prefill and decoding agree; decoding goes on across pages; the first tokens of a sequence come one by one."""
    toks, ref = want(name, 203, 0)
    rep = Replay(make_llm(folder, name, fmt, device))
    got = L.replay_one(rep, toks, [20] + [1] * 183)
    check_ok(device)
    assert_close(got, ref, fmt)
    assert_close(L.replay_one(rep, toks[:9], [1] * 9), ref[:9], fmt)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
@pytest.mark.parametrize("name", ["mixed", "wide", "odd"])
def test_batches_of_unequal_requests(folder, name, fmt, device):
    """Requests of unequal lengths in one batch, portions beside single tokens, one left out for some steps; the pool holds little more than
    what is live, so pages and slots are used again by later requests."""
    lens = {"a": 150, "b": 70, "c": 1, "d": 203, "e": 97, "f": 130}
    seq = {k: want(name, n, 0 if n == 203 else i + 1) for i, (k, n) in enumerate(lens.items())}
    llm = make_llm(folder, name, fmt, device, pages=10)
    rep = Replay(llm)
    at = {k: 0 for k in lens}
    got = {k: [] for k in lens}

    def step(**portions):
        entries = []
        for k, n in portions.items():
            n = min(n, lens[k] - at[k])
            entries.append({"id": k, "tokens": seq[k][0][at[k]: at[k] + n], "want": list(range(n))})
        out = rep.step(entries, [k for k, n in portions.items() if at[k] + n >= lens[k]])
        p = 0
        for e in entries:
            n = len(e["tokens"])
            got[e["id"]].append(out[p: p + n])
            at[e["id"]] += n
            p += n

    step(a=90, b=3)
    step(a=1, b=40, c=1)                       # c comes and goes
    for _ in range(5):
        step(a=1, b=1, d=2)
    step(a=30, d=100)                          # b is left out
    step(b=70, d=1)
    step(a=200, d=1)                           # a ends: its pages and slot go to e and f
    step(d=60, e=50, f=1)
    for _ in range(12):
        step(d=1, e=1, f=2)
    step(d=200, e=200, f=105)
    assert llm.blocks.num_free == 10 and sorted(llm._free_slots) == [0, 1, 2, 3] and not rep.live
    check_ok(device)
    for k in lens:
        assert at[k] == lens[k]
        assert_close(torch.cat(got[k]), seq[k][1], fmt, k)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_page_sizes_do_not_matter(folder, name, device):
    toks, ref = want(name, 203, 0)
    for page in (16, 128, 24):                 # 24 is no page size of the tcgen05 kernels
        got = L.replay_one(Replay(make_llm(folder, name, "bf16", device, pages=30, page=page)), toks, [101, 1, 1, 100])
        assert_close(got, ref, "bf16", page)
    check_ok(device)


@pytest.mark.gpu
@pytest.mark.parametrize("fmt", FORMATS)
def test_long_sequence(folder, fmt):
    """Several hundred tokens in large and small portions, then decoding far from the start; single layers of each kind see the whole of it."""
    toks, ref = want("wide", 700, 3)
    got = L.replay_one(Replay(make_llm(folder, "wide", fmt, "cuda")), toks, [520, 1, 1, 19, 100] + [1] * 59)
    check_ok("cuda")
    assert_close(got, ref, fmt)


@pytest.mark.parametrize("device", DEVICES)
def test_stream_after_every_layer(folder, device):
    toks = L.tokens(get_model("deep"), 75, 5)
    cap = []
    O.forward(get_model("deep"), toks, capture=cap)
    llm = make_llm(folder, "deep", "f32", device)
    llm.model.snapshot_layers = range(len(cap))
    Replay(llm).step([{"id": "x", "tokens": toks, "want": [74]}])
    assert len(cap) == 22 == len(llm.model.runs)
    for li, x in enumerate(cap):
        d = llm.model.snapshots[li].double().cpu() - x
        assert d.abs().max() < 2e-4 * x.abs().max(), li


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation_through_the_scheduler(folder, name, fmt, device):
    """``LLM.generate`` (continuous batching, chunked prompts, a pool too small for all at once) and the static-batch engine (CUDA graph on a
    GPU): each token is the reference's best, or within rounding of it."""
    model = get_model(name)
    prompts = [L.tokens(model, n, 20 + n) for n in (5, 90, 131)]
    new = 12
    llm = make_llm(folder, name, fmt, device, pages=6, slots=3, max_batch_tokens=48)
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=new))
    eng = Engine(weights(folder, name, fmt, device), max_batch=3, max_seq_len=256, page_size=PAGE, max_prefill_tokens=100)
    outs2 = eng.generate(prompts, SamplingParams(max_new_tokens=new))
    check_ok(device)
    for res in (outs, outs2):
        for p, o in zip(prompts, res):
            assert len(o) == new
            ref = O.forward(model, p + o)[len(p) - 1: -1]
            scale = (ref - ref.mean(-1, keepdim=True)).pow(2).mean().sqrt()
            gap = ref.max(-1).values - ref[torch.arange(new), torch.tensor(o)]
            assert (gap / scale).max() < 3 * TOL[fmt]
    assert llm.blocks.num_free == 6


@pytest.mark.parametrize("device", DEVICES)
def test_many_and_wide_heads(tmp_path, device):
    """More query heads per key head than an attention tile has rows, heads wider than the tcgen05 kernels take, latents of other sizes."""
    name = "heads"
    C.CASES[name] = (64, 50, 1e-2, 0.8, [C.attention(150, 1, 8, 8, 0.4, 0.3, 9, C.moe(3, 2, 16, 16)), C.latent(37, 16, 4, 12, 200, 1e3, 0.2, None), C.attention(2, 1, 136, 200, 0.1, 0.2, 30, None),
                                     C.latent(2, 150, 70, 130, 64, 1e3, 0.08, C.dense(40)), C.mingru(600, None)])
    try:
        model = C.make_model(name)
    finally:
        del C.CASES[name]
    C.save_model(model, str(tmp_path))
    toks = L.tokens(model, 90, 1)
    ref = O.forward(model, toks)
    for fmt in FORMATS:
        llm = LLM(loader.load_safetensors(str(tmp_path), fmt, device), None, max_running=4, num_pages=4, page_size=PAGE)
        assert_close(L.replay_one(Replay(llm), toks, [70, 1, 2, 17]), ref, fmt)
    check_ok(device)


def loud_model(name):
    """The model with larger queries and keys: single keys, some of them far away, rule the sums."""
    m = copy.deepcopy(get_model(name))
    for i, sp in enumerate(m["config"]["layers"]):
        if sp["type"] != "mingru":
            for c in ("q", "k", "uk"):
                if f"l{i}.mix.{c}" in m["t"]:
                    m["t"][f"l{i}.mix.{c}"] = m["t"][f"l{i}.mix.{c}"] * 2
    return m


def _every(m, delta):
    for sp in m["config"]["layers"]:
        if sp["type"] == "attention":
            sp["mixer"]["q_temp"]["every"] += delta


def _base(m):
    for sp in m["config"]["layers"]:
        if sp["type"] == "latent_attention":
            sp["mixer"]["rot"]["base"] *= 1.1


def _scaled(m, part, by):
    for k in m["t"]:
        if k.endswith(part):
            m["t"][k] = m["t"][k] * by


def _places(m):
    for k in m["t"]:
        if k.endswith(".dwa") and m["t"][k].numel() > 2:
            m["t"][k] = m["t"][k].clone()
            m["t"][k][[0, 1]] = m["t"][k][[1, 0]]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_what_single_mechanisms_change_shows(tmp_path, name, device):
    """A step of the temperature that is one off, another rotation, distance bias, shared expert's gate, residual factor, order of the averaged places or bias of a
    gate shows in these models far above the tolerance; prompts, portions and single tokens.  (In 32-bit: such scores make much of the rounding of keys to 16 bits.)"""
    model, fmt = loud_model(name), "f32"
    C.save_model(model, str(tmp_path))
    toks = L.tokens(model, 180, 7)
    ref = O.forward(model, toks)
    for change in (lambda m: _every(m, 1), _base, lambda m: _scaled(m, "mix.r1", 0.97), lambda m: _scaled(m, "mix.r2", 0.95), lambda m: _scaled(m, "shared.sg", 0.9),
                   lambda m: m["config"].update(residual_mult=m["config"]["residual_mult"] * 1.01), _places, lambda m: _scaled(m, "z.b", 0.98), lambda m: _scaled(m, "up.b", 0.9)):
        off = copy.deepcopy(model)
        change(off)
        assert L.err(O.forward(off, toks), ref).max() > 10 * TOL[fmt]
    w = loader.load_safetensors(str(tmp_path), fmt, device)
    for cut in ([180], [133, 2, 2, 3] + [1] * 40, L.cuts(180, [2, 31, 64, 1])):
        llm = LLM(w, None, max_running=4, num_pages=4, page_size=PAGE)
        assert L.err(L.replay_one(Replay(llm), toks, cut), ref).max() < 2 * TOL[fmt], cut[:3]
    check_ok(device)


@pytest.mark.parametrize("device", DEVICES)
def test_sampling_is_served(folder, device):
    llm = make_llm(folder, "mixed", "bf16", device)
    sp = SamplingParams(max_new_tokens=6, temperature=0.8, top_k=20, top_p=0.9, seed=3)
    a = llm.generate([L.tokens(get_model("mixed"), 30, 9)], sp)
    assert len(a[0]) == 6 and all(0 <= t < 211 for t in a[0])


@pytest.mark.gpu
@pytest.mark.parametrize("fmt,dtype", [("bf16", "bfloat16"), ("f32", "float32")])
def test_trace_program(folder, tmp_path, fmt, dtype):
    weights(folder, "wide", fmt, "cpu")
    toks, ref = want("wide", 203, 0)
    steps, at = [], 0
    for i, n in enumerate([100, 2, 1, 100]):
        steps.append({"step": i, "entries": [{"id": "q", "tokens": toks[at: at + n], "want": [] if i == 1 else [0, n - 1]}], "end": ["q"] if i == 3 else []})
        at += n
    prog = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, prog, "--model", os.path.join(str(folder), "wide"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "256"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    for i, rows in ((0, [0, 99]), (2, [102, 102]), (3, [103, 202])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4")).reshape(2, -1)
        assert_close(got, ref[rows], fmt)


# ------------------------------------------------------------------------------------------ configuration, loading, command line
def test_config_reads_every_size(folder):
    cfg = weights(folder, "mixed", "f32", "cpu").cfg
    assert (cfg.arch, cfg.vocab, cfg.hidden, cfg.rms_eps, cfg.norm_kind, cfg.norm_offset, cfg.residual_mult, cfg.depth_average) == ("zedirax", 211, 136, 1e-2, "rms", 1.0, 0.6, True)
    assert (cfg.tie_embeddings, cfg.embed_scale, cfg.logit_scale, cfg.loop, cfg.parallel_ffn, cfg.post_norm) == (False, 1.0, 1.0, None, False, False)
    u, a, x = cfg.layer_specs[:3]
    assert (u.mixer, u.n_heads, u.head_dim, u.v_dim, u.has_state) == ("mingru", 1, 1, 200, True)
    assert (u.moe.n_experts, u.moe.top, u.moe.ffn, u.moe.shared, u.moe.act, u.moe.gated, u.moe.renorm, u.moe.groups, u.moe.router) == (10, 3, 48, 72, "gelu", False, True, 1, "softmax")
    assert (a.mixer, a.n_heads, a.n_kv_heads, a.head_dim, a.v_dim, a.scale, a.log_bias, a.temp_coef, a.temp_every, a.qkv_bias, a.qk_unit) == ("attention", 6, 3, 40, 24, 0.25, True, 0.3, 17, False, False)
    assert (a.ffn, a.act, a.ffn_bias, a.moe) == (200, "gelu_tanh", True, None)
    assert (x.mixer, x.n_heads, x.head_dim, x.rot_dim, x.v_dim, x.kv_rank, x.q_rank, x.scale, x.out_gate, x.sink) == ("latent", 3, 24, 8, 40, 72, 0, 0.2, True, False)
    assert (x.rotary.dims, x.rotary.base, x.rotary.factor, x.rotary.halves, x.moe.shared) == (8, 1e4, 0.0, True, 0)
    assert [sp.has_ffn for sp in cfg.layer_specs] == [True, True, True, False, False, True]
    assert cfg.has_recurrent_state and ModelConfig(**cfg.to_dict()).layer_specs == cfg.layer_specs


def test_saved_checkpoints_load_again(tmp_path):
    from gemm_b200.models.weights import RandomSource, build_weights
    cfg = get_config("tiny-zedirax")
    loader.save_hf_checkpoint(cfg, RandomSource(cfg, seed=4, device="cpu"), str(tmp_path))
    a, b = loader.load_safetensors(str(tmp_path), "bf16", "cpu"), build_weights(cfg, RandomSource(cfg, seed=4, device="cpu"), "bf16", "cpu")
    assert a.cfg == b.cfg and torch.equal(a.embed, b.embed) and torch.equal(a.lm_head.w, b.lm_head.w)
    for x, y in zip(a.layers, b.layers):
        assert all(torch.equal(p.w, q.w) for p, q in zip(x.linears(), y.linears()))
        assert torch.equal(x.depth_w, y.depth_w) and (x.log_bias is None or torch.equal(x.log_bias, y.log_bias)) and (x.sh_dot is None or torch.equal(x.sh_dot, y.sh_dot))
        assert all(torch.equal(p.bias, q.bias) for p, q in zip(x.linears(), y.linears()) if p.bias is not None)
    out = LLM(a, None, num_pages=4, page_size=64).generate([[1, 2, 3]], SamplingParams(max_new_tokens=3))
    assert len(out[0]) == 3


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][1].update(type="spiral"), "spiral"),
    (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "sparse"),
    (lambda c: c.update(architecture="Unheard"), "Unheard"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=6), "rotation"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=11), "experts per token"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=40), "l0.mlp.e0.up"),
    (lambda c: c["layers"][0]["mixer"].update(width=100), "l0.mix"),
])
def test_unknown_parts_are_refused(tmp_path, change, word):
    m = copy.deepcopy(get_model("mixed"))
    change(m["config"])
    C.save_model(m, str(tmp_path))
    with pytest.raises(ValueError, match=word):
        LLM(loader.load_safetensors(str(tmp_path), "f32", "cpu"), None, num_pages=2, page_size=64)


def test_a_missing_or_misshapen_tensor_is_named(tmp_path):
    m = copy.deepcopy(get_model("mixed"))
    del m["t"]["l2.mlp.e3.up"]
    C.save_model(m, str(tmp_path / "a"))
    with pytest.raises(ValueError, match="l2.mlp.e3.up"):
        loader.load_safetensors(str(tmp_path / "a"), "f32", "cpu")
    m = copy.deepcopy(get_model("mixed"))
    m["t"]["l3.dwa"] = m["t"]["l3.dwa"][:-1]
    C.save_model(m, str(tmp_path / "b"))
    with pytest.raises(ValueError, match="l3.dwa"):
        loader.load_safetensors(str(tmp_path / "b"), "f32", "cpu")


@pytest.mark.parametrize("device", DEVICES)
def test_command_line(folder, device):
    model = get_model("mixed")
    weights(folder, "mixed", "f32", "cpu")
    p = L.tokens(model, 40, 2)
    r = subprocess.run([sys.executable, "-m", "gemm_b200", "generate", "--model", os.path.join(str(folder), "mixed"), "--format", "f32", "--device", device,
                        "--ids", "--prompt", " ".join(map(str, p)), "--max-new-tokens", "4", "--pages", "8", "--page-size", "64"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr
    out = [int(x) for x in r.stdout.replace(",", " ").replace("[", " ").replace("]", " ").split() if x.isdigit()][-4:]
    ids = list(p)
    for t in out:
        assert int(O.forward(model, ids)[-1].argmax()) == t
        ids.append(t)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("fmt", FORMATS)
def test_saved_inference_state_goes_on(folder, tmp_path, fmt, device):
    """Keys and values, latents and recurrent states written to a file and read by another engine with other page numbers."""
    from gemm_b200.utils import checkpoint
    w = weights(folder, "mixed", fmt, device)
    prompts = [torch.tensor(L.tokens(get_model("mixed"), n, n), dtype=torch.int32) for n in (70, 7)]
    a = Engine(w, max_batch=2, max_seq_len=160, page_size=PAGE)
    first = a._sample(a.prefill(prompts, reserve=8), SamplingParams(), 0)
    path = str(tmp_path / "state")
    checkpoint.save_state(a, path, first)
    a.begin_decode(first, SamplingParams(), 6, use_graph=False)
    ref = [a.decode_step().cpu().tolist() for _ in range(4)]
    b = Engine(w, max_batch=2, max_seq_len=160, page_size=PAGE, num_pages=9)
    b.pages.alloc(3)
    nxt = checkpoint.load_state(b, path)
    b.begin_decode(nxt, SamplingParams(), 6, use_graph=False)
    assert [b.decode_step().cpu().tolist() for _ in range(4)] == ref


def test_recurrent_models_refuse_speculation(folder):
    from gemm_b200.serve.speculative import NgramDrafter
    with pytest.raises(ValueError, match="recurrent"):
        make_llm(folder, "mixed", "f32", "cpu").set_drafter(NgramDrafter(gamma=2))
