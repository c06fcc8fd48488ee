"""Bepepel through the engine against the plain implementation.

Replays through bin/trace_run: the same requests whole, with their last tokens one by one, in
portions of changing size down to two tokens, and mixed (up to four live, portions beside single
tokens, few pages and four state slots so that both are used again, freed pages filled with NaN),
in float32 and bfloat16, also from captured CUDA graphs.  "Sharp" variants scale the scores and
lengthen the memories so that a lost far key, a kept first key left out, a key on the wrong side of a
window's edge or a lost state shows.  The stream after every layer.  Generation through LLMEngine,
ContinuousBatchingEngine and the command line.  The kernels and parts one by one."""
import copy
import math
from types import SimpleNamespace

import pytest
import torch

import bepepel_util as bu
import plain_bepepel as plain
import replay_util as ru

pytestmark = pytest.mark.gpu

LENGTHS = {"mix": [1, 9, 40, 131, 260], "odd": [2, 17, 64, 150], "wide": [3, 33, 97, 230], "long": [4, 299, 345, 705]}

# gap of router logits below which the engine's arithmetic may send a token to another expert
CLOSE_CALL = {"bfloat16": 0.06, "float32": 1e-5}


def first_close_call(config, weights, ids, dtype):
    """(logits, first position at which the plain router's choice hangs on less than CLOSE_CALL)."""
    plain.ROUTING_MARGINS = []
    try:
        logits = plain.forward(config, weights, ids)[0].float()
        close = [t for t, m in plain.ROUTING_MARGINS if m < CLOSE_CALL[dtype]]
    finally:
        plain.ROUTING_MARGINS = None
    return logits, (min(close) if close else len(ids))


def rounded_inputs(config, weights, ids, monkeypatch):
    """The plain logits when every sublayer's input is rounded to bfloat16: how far one rounding alone moves
    each position (a head or a group that is divided by a small root mean square magnifies it)."""
    exact = plain.layer_norm
    with monkeypatch.context() as m:
        m.setattr(plain, "layer_norm", lambda *a: exact(*a).bfloat16().double())
        return plain.forward(config, weights, ids)[0].float()


def replay(name, dtype, tmp_path, monkeypatch, cuda_graph=False, sharp=False):
    """Every position within rounding, up to the first position of a request at which the plain router's
    choice of experts is a close call; from there on (that token may have had another expert, and the
    tokens after it see it) finite and of the logits' size.  The same configurations with every expert
    chosen leave the router no choice and are held to the rounding bound everywhere (tests below)."""
    spec = bu.CONFIGS[name]
    model_dir = str(tmp_path / "model")
    config, weights = bu.make_folder(model_dir, name, sharp=sharp)
    prompts = {f"p{n}": ru.random_ids(n, config["vocab"], 100 + n) for n in LENGTHS[name.split("_")[0]]}
    trace, peak = ru.build_four_mode_trace(prompts, spec["page_size"])
    got = ru.run_trace(model_dir, dtype, trace, peak, str(tmp_path / "out"), page_size=spec["page_size"],
                       cuda_graph=cuda_graph, max_requests=4)
    refs = {n: first_close_call(config, weights, ids, dtype) for n, ids in prompts.items()}
    moved = {n: (rounded_inputs(config, weights, ids, monkeypatch) - refs[n][0]).abs().amax(-1) if dtype == "bfloat16" else None
             for n, ids in prompts.items()}
    modes, strict = set(), 0
    for (step, rid, pos), row in got.items():
        mode, pname = rid.split("/")
        modes.add(mode.rstrip("01"))
        ref = refs[pname][0][pos]
        assert torch.isfinite(row).all(), (step, rid, pos)
        err = (row - ref).abs().max().item()
        scale = max(ref.abs().max().item(), 1e-3)
        if pos < refs[pname][1]:
            strict += 1
            bound = (1e-3 if sharp else 1e-4) * max(scale, 1.0) if dtype == "float32" \
                else 0.04 * scale + 0.02 + 3.0 * float(moved[pname][pos])
            assert err <= bound, f"first wrong place: step {step} request {rid} position {pos}: {err} (scale {scale})"
        else:
            assert err <= 2.0 * scale + 0.5, (step, rid, pos, err)
    assert modes == {"whole", "tail", "portions", "mixed"}
    assert dtype != "float32" or strict >= 0.5 * len(got)  # in 32-bit, close calls are the exception
    return strict / max(len(got), 1)


def with_every_expert_chosen(name):
    """``top`` equals the number of experts: logits, weights, the experts' products and their sum all
    run, and no logit decides anything."""
    spec = copy.deepcopy(bu.CONFIGS[name])
    for e in spec["config"]["layers"]:
        if e.get("mlp") and e["mlp"]["kind"] == "moe":
            e["mlp"]["router"]["top"] = e["mlp"]["router"]["experts"]
    bu.CONFIGS[name + "_every_expert"] = spec
    return name + "_every_expert"


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "long"])
def test_replay_float32(name, tmp_path, monkeypatch):
    replay(name, "float32", tmp_path, monkeypatch)


@pytest.mark.parametrize("name", ["mix", "odd"])
def test_replay_bfloat16(name, tmp_path, monkeypatch):
    replay(name, "bfloat16", tmp_path, monkeypatch)


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "long"])
def test_replay_bfloat16_without_routing_is_within_rounding_everywhere(name, tmp_path, monkeypatch):
    assert replay(with_every_expert_chosen(name), "bfloat16", tmp_path, monkeypatch) == 1.0


@pytest.mark.parametrize("name", ["mix", "wide"])
def test_replay_bfloat16_single_token_steps_from_captured_graphs(name, tmp_path, monkeypatch):
    replay(with_every_expert_chosen(name), "bfloat16", tmp_path, monkeypatch, cuda_graph=True)


@pytest.mark.parametrize("name", ["mix", "odd", "long"])
def test_replay_float32_sharp_keys_and_long_memories(name, tmp_path, monkeypatch):
    replay(name, "float32", tmp_path, monkeypatch, sharp=True)


# ------------------------------------------------------------------ the stream after every layer
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name in ("mix", "odd", "wide", with_every_expert_chosen("mix"), with_every_expert_chosen("wide")):
        d = str(tmp_path_factory.mktemp(f"bepepel_{name}"))
        out[name] = (d,) + bu.make_folder(d, name)
    return out


def load(folder, dtype):
    from dispec_b200 import load_model
    return load_model(folder, dtype, "cuda:0")


@pytest.mark.parametrize("name", ["mix", "odd", "wide"])
def test_stream_after_every_layer_float32(folders, name):
    from dispec_b200.engine import ModelRunner, SeqEntry
    from dispec_b200.engine.batch import build_context
    folder, config, weights = folders[name]
    model = load(folder, "float32")
    r = ModelRunner(model, page_size=bu.CONFIGS[name]["page_size"], num_pages=16, max_num_seqs=2)
    ids = ru.random_ids(37, config["vocab"], 7)
    r.admit("a")
    r.cache.extend("a", len(ids))
    ctx, _ = build_context([SeqEntry("a", ids, 0, [])], r.cache, r.storage, r.states, r.staging, r.dtype, r.device,
                           model.attention_tile_tokens, r.vocab_size)
    ctx.layer_trace = []
    with torch.inference_mode():
        model.forward(ctx)
    want = []
    plain.forward(config, weights, ids, layer_trace=want)
    assert len(ctx.layer_trace) == len(want) == len(config["layers"])
    for i, (got, ref) in enumerate(zip(ctx.layer_trace, want)):
        assert (got.cpu().double() - ref).abs().max() < 1e-4 * max(1.0, ref.abs().max().item()), f"layer {i}"


# ------------------------------------------------------------------ generation entry points
def assert_greedy(weights, config, prompt, got, dtype):
    """Teacher-forced on the engine's tokens: each equals the plain argmax, or the plain top-2 gap
    there is below what the type can resolve."""
    logits = plain.forward(config, weights, list(prompt) + list(got))[0].float()
    for i, tok in enumerate(got):
        row = logits[len(prompt) - 1 + i]
        top2 = torch.topk(row, 2)
        reach = 1e-4 if dtype == "float32" else 2 * (0.03 * row.abs().max().item() + 0.02)
        assert tok == int(top2.indices[0]) or float(top2.values[0] - top2.values[1]) < reach, (i, tok)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_llm_engine(folders, dtype):
    from dispec_b200 import LLMEngine, SamplingParams
    folder, config, weights = folders["mix" if dtype == "float32" else "mix_every_expert"]
    engine = LLMEngine(load(folder, dtype), num_blocks=32, cuda_graph=dtype == "bfloat16")
    for n in (1, 9, 40):  # the same engine: pages and slots are used again
        prompt = ru.random_ids(n, config["vocab"], 300 + n)
        got = engine.generate(prompt, 10, SamplingParams(temperature=0.0))
        assert len(got) == 10
        assert_greedy(weights, config, prompt, got, dtype)
    cache = engine.runner.cache
    assert all(cache.num_free_pages(g) == 32 for g in range(len(cache.groups)))


def test_long_decoding_float32_past_every_window(folders):
    from dispec_b200 import LLMEngine, SamplingParams
    folder, config, weights = folders["odd"]
    engine = LLMEngine(load(folder, "float32"), num_blocks=32)
    prompt = ru.random_ids(3, config["vocab"], 1)
    got = engine.generate(prompt, 150, SamplingParams())
    assert len(got) == 150
    assert_greedy(weights, config, prompt, got, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_continuous_batching_more_requests_than_slots(folders, dtype):
    """Seven requests through three slots and a small pool: portions of prompts beside decoded
    tokens; slots, states and pages of finished requests go to waiting ones."""
    from dispec_b200 import ContinuousBatchingEngine, KVConfig, SamplingParams
    folder, config, weights = folders["wide" if dtype == "float32" else "wide_every_expert"]
    engine = ContinuousBatchingEngine(load(folder, dtype), KVConfig(block_size=32), num_blocks=24,
                                      max_batch_tokens=48, chunk_size=20, max_num_seqs=3)
    reqs = []
    for i, n in enumerate([1, 9, 40, 64, 9, 70, 2]):
        prompt = ru.random_ids(n, config["vocab"], 400 + i)
        reqs.append((engine.add_request(prompt, 9, SamplingParams(temperature=0.0)), prompt))
    engine.run_until_done()
    out = engine.collect_outputs()
    for rid, prompt in reqs:
        assert len(out[rid]) == 9
        assert_greedy(weights, config, prompt, out[rid], dtype)
    assert engine.runner.cache.free_slots() == 3


def test_command_line_serves_a_folder_and_a_configuration_with_random_weights(tmp_path):
    """`python -m dispec_b200 generate` on a Bepepel folder (whose rank only the tensors give): greedy
    tokens equal the plain ones; `random` writes a folder for the same configuration that `generate`
    serves too."""
    import json
    import os
    import subprocess
    import sys
    folder = str(tmp_path / "model")
    config, weights = bu.make_folder(folder, "odd")
    env = dict(os.environ, PYTHONPATH=ru.ROOT)
    prompts = [[5, 17, 3, 90], list(range(7, 33))]
    cmd = [sys.executable, "-m", "dispec_b200", "generate", "--dtype", "float32", "--max-new", "8", "--block-size", "8",
           "--num-blocks", "48", "--max-batch-tokens", "16", "--chunk-size", "6"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(map(str, p))]
    proc = subprocess.run(cmd + ["--model", folder], check=True, env=env, cwd=ru.ROOT, capture_output=True, text=True)
    lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
    assert [ln["prompt_tokens"] for ln in lines] == [len(p) for p in prompts]
    for ln, prompt in zip(lines, prompts):
        assert len(ln["output_ids"]) == 8
        assert_greedy(weights, config, prompt, ln["output_ids"], "float32")
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(config))
    made = str(tmp_path / "made")
    subprocess.run([sys.executable, "-m", "dispec_b200", "random", "--config", str(cfg_path), "--out", made, "--seed", "5",
                    "--std", "0.08"], check=True, env=env, cwd=ru.ROOT)
    from safetensors.torch import load_file
    made_weights = {k: v.float() for k, v in load_file(os.path.join(made, "model.safetensors")).items()}
    assert {k: tuple(v.shape) for k, v in made_weights.items()} == plain.tensor_shapes(config)
    proc = subprocess.run(cmd + ["--model", made], check=True, env=env, cwd=ru.ROOT, capture_output=True, text=True)
    lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
    for ln, prompt in zip(lines, prompts):
        assert_greedy(made_weights, config, prompt, ln["output_ids"], "float32")


# ----------------------------------------------------------------------- kernels one by one
def dev(t, dtype=torch.float32):
    return t.to(device="cuda:0", dtype=dtype).contiguous()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda:0")


def step_arrays(portions):
    """``portions``: (slot, first position, tokens) of each request -> the step's arrays.  A first position of
    -1 makes a padding row."""
    pos, seq, start = [], [], [0]
    for s, (_, first, n) in enumerate(portions):
        pos += [-1] * n if first < 0 else list(range(first, first + n))
        seq += [s] * n
        start.append(start[-1] + n)
    return SimpleNamespace(positions=i32(pos), seq_of_token=i32(seq), q_start=i32(start),
                           state_slot=i32([p[0] for p in portions]))


@pytest.mark.parametrize("width,copies", [(52, False), (256, True), (1000, True)])
def test_scaled_pre_norm_block_sums_and_hands_on_the_next_norm(width, copies):
    """The block with stand-in sublayers: x + m f(N1(x)), then + m g(N2(.)), norms with gain and bias."""
    from dispec_b200.parts.base import WideStream
    from dispec_b200.parts.block import LayerNormTail, ScaledPreNormBlock
    from dispec_b200.parts.norms import LayerNorm32
    g = torch.Generator().manual_seed(width)
    x = torch.randn(6, width, generator=g) * 3 + 0.7
    dtype = torch.bfloat16 if copies else torch.float32
    norms, wb = [], []
    for _ in range(3):
        w, b = 1 + 0.2 * torch.randn(width, generator=g), 0.3 * torch.randn(width, generator=g)
        n = LayerNorm32(width, 1e-5, with_bias=True)
        n.load({"weight": dev(w), "bias": dev(b)})
        norms.append(n)
        wb.append((w.double(), b.double()))

    class Sub:
        def __init__(self, f):
            self.f = f

        def forward(self, ctx, h, *rest):
            assert h.dtype == dtype
            return self.f(h.float())

    block = ScaledPreNormBlock(width, 0.37, norms[0], Sub(lambda h: h * 0.5 + 1.0), norms[1], Sub(torch.tanh))
    s, ctx = WideStream(dev(x), None), SimpleNamespace(dtype=dtype)
    out, nxt = block.forward(ctx, s, None, None, None, then_norm=LayerNormTail(norms[2].weight, 1e-5, norms[2].bias))
    rnd = lambda t: t.to(dtype).double()
    x1 = x.double() + 0.37 * (rnd(plain.layer_norm(x.double(), *wb[0], 1e-5)) * 0.5 + 1.0)
    x2 = x1 + 0.37 * torch.tanh(rnd(plain.layer_norm(x1, *wb[1], 1e-5)))
    tol = 0.02 if copies else 1e-5
    assert out is s and (s.full.cpu().double() - x2).abs().max() < tol
    want = plain.layer_norm(s.full.cpu().double(), *wb[2], 1e-5)
    assert nxt.dtype == dtype and (nxt.cpu().double() - want).abs().max() < (0.02 if copies else 1e-5) * want.abs().max()
    # rows picked out, as the final norm does it
    rows = i32([4, 0])
    got = norms[2].forward(ctx, s, rows=rows).cpu().double()
    assert (got - want[[4, 0]]).abs().max() < (0.02 if copies else 1e-5) * want.abs().max()
    assert block.forward(ctx, s, nxt, None, None)[1] is None  # the last block keeps nothing pending


@pytest.mark.parametrize("groups,per", [(3, 10), (2, 96), (1, 640), (5, 33)])
def test_norm_of_gated_groups_with_a_gain_per_channel(groups, per):
    from dispec_b200.ops import norm32
    g = torch.Generator().manual_seed(per)
    T, n = 7, groups * per
    y, z, w = torch.randn(T, n, generator=g), torch.randn(T, n + 9, generator=g), torch.randn(n, generator=g)
    out = torch.full((T, n + 6), float("nan"), device="cuda:0")
    norm32.head_norm_gate(dev(y), groups, 1e-5, torch.float32, gain=dev(w), gate=dev(z)[:, 4:4 + n], gate_first=True,
                          out=out[:, 3:3 + n])
    want = plain.gated_group_norm(y.double(), z[:, 4:4 + n].double(), w.double(), groups, 1e-5)
    assert (out[:, 3:3 + n].cpu().double() - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item())
    assert torch.isnan(out[:, :3]).all() and torch.isnan(out[:, 3 + n:]).all()


@pytest.mark.parametrize("dtype,T,W,ff", [(torch.float32, 9, 52, 30), (torch.bfloat16, 9, 64, 96), (torch.bfloat16, 90, 128, 64),
                                          (torch.bfloat16, 200, 256, 512), (torch.bfloat16, 1, 1024, 64), (torch.bfloat16, 5, 64, 40)])
def test_gelu_unit_in_every_form_of_the_gate_up_product(dtype, T, W, ff):
    """The 32-bit path, the few-row product (also with K split), the many-row product, and widths that
    none of them fuses; gates from far below to far above zero."""
    from dispec_b200.parts.swiglu import SwiGLUFeedForward
    g = torch.Generator().manual_seed(W + T)
    P = {n: (torch.randn((W, ff) if n == "down" else (ff, W), generator=g) / W ** 0.5).bfloat16().float() for n in ("gate", "up", "down")}
    P["gate"] *= 4.0
    h = torch.randn(T, W, generator=g).bfloat16().float()
    part = SwiGLUFeedForward(W, ff, out_float32=True, act="gelu_tanh")
    part.load({n + "_proj.weight": dev(P[n], dtype) for n in P})
    got = part.forward(SimpleNamespace(dtype=dtype), dev(h, dtype)).cpu().double()
    want = plain.glu(h.double(), {"m." + n: t.double() for n, t in P.items()}, "m.", plain.gelu_tanh)
    assert torch.isfinite(got).all()
    assert (got - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.03) * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("E,top", [(6, 3), (9, 1), (16, 16), (40, 8), (1, 1)])
def test_router_kernel_weighs_the_chosen_logits_with_a_bias(E, top):
    from dispec_b200.ops import moe
    g = torch.Generator().manual_seed(E + top)
    T, W = 41, 29
    h, w, b = torch.randn(T, W, generator=g), 3 * torch.randn(E, W, generator=g), torch.randn(E, generator=g)
    h[5] *= 20.0  # logits hundreds apart: the others' weights underflow to 0, nothing else happens
    ids, wts = moe.route(dev(h), dev(w), 1, 1, top, score="chosen_softmax", bias=dev(b))
    want_ids, want_w = plain.route(h.double(), {"r.router": w.double(), "r.router.b": b.double()}, "r.", {"experts": E, "top": top})
    for t in range(T):
        assert ids[t].tolist() == want_ids[t].tolist(), t  # by falling logit
        assert (wts[t].cpu().double() - want_w[t]).abs().max() < 3e-5
        assert abs(float(wts[t].sum()) - 1.0) < 1e-5


@pytest.mark.parametrize("dtype,W,ff", [(torch.float32, 52, 14), (torch.bfloat16, 64, 24)])
@pytest.mark.parametrize("shared", [True, False])
def test_mixture_part_with_a_biased_router(dtype, W, ff, shared):
    from dispec_b200.parts.moe import GatedMoE
    from dispec_b200.parts.swiglu import SwiGLUFeedForward
    g = torch.Generator().manual_seed(W)
    E, top, T = 6, 2, 45
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": E, "top": top}}
    if shared:
        mlp["shared"] = {"ff": ff + 8}
    shapes = {"router": (E, W), "router.b": (E,), "shared.gate": (ff + 8, W), "shared.up": (ff + 8, W), "shared.down": (W, ff + 8)}
    for e in range(E):
        shapes.update({f"e{e}.{n}": (W, ff) if n == "down" else (ff, W) for n in ("gate", "up", "down")})
    P = {"m." + n: (torch.randn(s, generator=g) * (3.0 if n == "router" else 1.0) / s[-1] ** 0.5).bfloat16().float() for n, s in shapes.items()}
    h = torch.randn(T, W, generator=g).bfloat16().float()
    unit = SwiGLUFeedForward(W, ff + 8, out_float32=True)
    unit.load({n + "_proj.weight": dev(P["m.shared." + n], dtype) for n in ("gate", "up", "down")})
    part = GatedMoE(W, ff, E, top, None, alpha=1.0, up_shift=0.0, score="chosen_softmax", weight_on="output", router_bias=True,
                    shared=unit if shared else None)
    tensors = {"router.weight": dev(P["m.router"]), "router.bias": dev(P["m.router.b"])}
    for e in range(E):
        for n in ("gate", "up", "down"):
            tensors[f"experts.{e}.{n}.weight"] = dev(P[f"m.e{e}.{n}"], dtype)
    part.load(tensors)
    got = part.forward(SimpleNamespace(dtype=dtype), dev(h, dtype)).cpu().double()
    want = plain.moe(h.double(), {k: v.double() for k, v in P.items()}, "m.", mlp)
    assert (got - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.03) * max(1.0, want.abs().max().item())


# ----------------------------------------------------------------------- short convolutions
@pytest.mark.parametrize("taps,channels,heads", [(1, 10, 3), (2, 37, 2), (4, 1100, 24), (5, 64, 1), (9, 12, 5)])
def test_conv_kernel_carries_its_inputs_from_portion_to_portion(taps, channels, heads):
    """Three requests in slots of a larger buffer, in steps of portions shorter and longer than the taps
    beside single tokens and padding rows; a slot whose request ended is zeroed and used again."""
    from dispec_b200.ops import short_conv as SC
    g = torch.Generator().manual_seed(taps * channels)
    cols, off = channels + heads + 7, 5
    w, b = torch.randn(channels, taps, generator=g), torch.randn(channels, generator=g)
    dtb, alog = torch.randn(heads, generator=g), torch.randn(heads, generator=g)
    lens = {2: 40, 0: 23, 3: 31}  # slot -> tokens
    u = {s: torch.randn(n, cols, generator=g) for s, n in lens.items()}
    u[2][7, off + channels] = 60.0  # a step size far in softplus' linear part
    hist = torch.full((5, taps - 1, channels), float("nan"), device="cuda:0")
    for s in lens:
        hist[s].zero_()
    done = {s: 0 for s in lens}
    got = {s: [] for s in lens}
    got_steps = {s: [] for s in lens}
    sizes = [(2, 1, 3), (1, 1, 1), (3, 2, 1), (7, 1, 12), (1, 5, 2), (40, 40, 40)]
    for k, step in enumerate(sizes):
        portions, rows = [], []
        for s, n in zip(lens, step):
            n = min(n, lens[s] - done[s])
            if n:
                portions.append((s, done[s], n))
                rows.append(u[s][done[s]:done[s] + n])
        if k % 2:  # a padding row names a slot that belongs to someone else
            portions.append((2, -1, 1))
            rows.append(torch.full((1, cols), 1e6))
        ctx = step_arrays(portions)
        out, steps = SC.conv_steps(dev(torch.cat(rows)), off, dev(w.t()), dev(b), hist if taps > 1 else None, ctx,
                                   step_offset=off + channels, step_bias=dev(dtb), a_log=dev(alog))
        at = 0
        for s, first, n in portions:
            if first >= 0:
                got[s].append(out[at:at + n].cpu())
                got_steps[s].append(steps[at:at + n].cpu())
                done[s] += n
            at += n
    assert done == lens
    for s in lens:
        y, kept = plain.short_conv(u[s][:, off:off + channels].double(), w.double(), torch.zeros(taps - 1, channels, dtype=plain.F))
        want = plain.silu(y + b.double())
        assert (torch.cat(got[s]).double() - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item())
        if taps > 1:
            assert (hist[s].cpu().double() - kept).abs().max() < 1e-6
        dt = plain.softplus(u[s][:, off + channels:off + channels + heads].double() + dtb.double())
        steps = torch.cat(got_steps[s]).double()
        assert ((steps[:, 0] - dt).abs() / (1 + dt)).max() < 1e-5
        assert (steps[:, 1] - torch.exp(-torch.exp(alog.double()) * dt)).abs().max() < 1e-5
    if taps > 1:
        assert torch.isnan(hist[1]).all() and torch.isnan(hist[4]).all()


@pytest.mark.parametrize("taps", [0, 1, 2, 4, 6])
@pytest.mark.parametrize("H,G,dk,dv,rot,interleaved,norm,pool", [
    (4, 2, 16, 8, 8, True, True, torch.float32), (5, 5, 6, 10, 6, True, True, torch.float32),
    (8, 2, 64, 128, 64, False, True, torch.bfloat16), (2, 1, 12, 4, 0, True, False, torch.float32)])
def test_conv_rotate_store_kernel(taps, H, G, dk, dv, rot, interleaved, norm, pool):
    """Convolution, rotation, norm and pages of two requests in portions down to one token, with a padding
    row; nothing but the tokens' own places in the pools is written."""
    from dispec_b200.ops import short_conv as SC
    g = torch.Generator().manual_seed(H * dk + taps)
    channels, page = (H + G) * dk + G * dv, 4
    w = torch.randn(channels, max(taps, 1), generator=g)
    if taps == 0:
        w = torch.ones(channels, 1)
    freq = torch.tensor([0.9 ** i for i in range(rot // 2)])
    lens = [21, 14]
    u = [torch.randn(n, channels, generator=g) for n in lens]
    tables = [[3, 0, 9, 7, 1, 12], [5, 2, 11, 8, -1, -1]]
    k_pool = torch.full((14, G, page, dk), float("nan"), dtype=pool, device="cuda:0")
    v_pool = torch.full((14, G, page, dv), float("nan"), dtype=pool, device="cuda:0")
    hist = torch.zeros(3, taps - 1, channels, device="cuda:0") if taps > 1 else None
    slots, done, got = [2, 0], [0, 0], [[], []]
    for step in ((2, 1), (1, 3), (5, 1), (1, 1), (30, 30)):
        portions, rows, who = [], [], []
        for s in range(2):
            n = min(step[s], lens[s] - done[s])
            if n:
                portions.append((slots[s], done[s], n))
                rows.append(u[s][done[s]:done[s] + n])
                who.append(s)
        portions.append((slots[0], -1, 1))
        rows.append(torch.full((1, channels), 1e6))
        ctx = step_arrays(portions)
        cache = SimpleNamespace(key_pool=k_pool, value_pool=v_pool, page_table=i32([tables[s] for s in who] + [[-1] * 6]), write=True)
        q = SC.qkv_conv_rotate_store(dev(torch.cat(rows)), dev(w.t()) if taps else None, hist, ctx, cache, dev(freq) if rot else None,
                                     rot, interleaved, H, G, dk, dv, pool, norm, 1e-5, value_scale=1.7)
        at = 0
        for s, (_, _, n) in zip(who, portions):
            got[s].append(q[at:at + n].cpu().double())
            done[s] += n
            at += n
    from dispec_b200.ops import library
    assert library.device_error() == 0
    tol = 1e-5 if pool == torch.float32 else 0.02
    for s in range(2):
        y, kept = plain.short_conv(u[s].double(), w.double(), torch.zeros(w.shape[1] - 1, channels, dtype=plain.F))
        pos = torch.arange(lens[s])
        q, k, v = y[:, :H * dk].view(-1, H, dk), y[:, H * dk:(H + G) * dk].view(-1, G, dk), y[:, (H + G) * dk:].view(-1, G, dv)
        if rot and not interleaved:  # the other pair layout, by a permutation of the dimensions
            perm = [i // 2 + (i % 2) * (rot // 2) for i in range(rot)] + list(range(rot, dk))
            inv = [perm.index(i) for i in range(dk)]
            q, k = (plain.turn_pairs(x[..., perm], pos, freq.double())[..., inv] for x in (q, k))
        elif rot:
            q, k = plain.turn_pairs(q, pos, freq.double()), plain.turn_pairs(k, pos, freq.double())
        if norm:
            q, k = plain.rms(q, 1e-5), plain.rms(k, 1e-5)
        assert (torch.cat(got[s]).view(-1, H, dk) - q).abs().max() < tol * q.abs().max()
        for t in range(lens[s]):
            pg, o = tables[s][t // page], t % page
            assert (k_pool[pg, :, o].cpu().double() - k[t]).abs().max() < tol * k.abs().max()
            assert (v_pool[pg, :, o].cpu().double() - 1.7 * v[t]).abs().max() < tol * 1.7 * v.abs().max()
        if taps > 1:
            assert (hist[slots[s]].cpu().double() - kept).abs().max() < 1e-6
    assert int(torch.isfinite(k_pool[:, 0, :, 0].float()).sum()) == sum(lens)


# ----------------------------------------------------------------------- recurrences
def recurrence_steps(lens, sizes):
    """Steps over requests of ``lens`` tokens in portions of ``sizes`` (one row of sizes a step)."""
    done, k = [0] * len(lens), 0
    while any(d < n for d, n in zip(done, lens)):
        step = []
        for s, n in enumerate(lens):
            c = min(sizes[k % len(sizes)][s], n - done[s])
            if c:
                step.append((s, done[s], c))
                done[s] += c
        yield step
        k += 1


SIZES = [(2, 1), (1, 1), (17, 1), (1, 40), (3, 2), (64, 8), (1, 1)]
DIMS = [(2, 6, 10), (3, 32, 70), (1, 48, 33), (2, 128, 16), (2, 100, 24), (1, 200, 12), (1, 300, 9)]


@pytest.mark.parametrize("H,d,dv", DIMS)
@pytest.mark.parametrize("rank,dtype", [(16, torch.float32), (5, torch.float32), (3, torch.bfloat16)])
def test_recurrence_with_a_decay_per_key_channel(H, d, dv, rank, dtype):
    """Portions, single tokens and padding rows against one plain scan; memories of hundreds of tokens.  The
    state after the last token too."""
    from dispec_b200.ops import recurrence as R
    g = torch.Generator().manual_seed(d + rank)
    lens, slots = [150, 90], [3, 1]
    cols = 2 * H * d + H * dv + rank + 3
    proj = [torch.randn(n, cols, generator=g).to(dtype) for n in lens]
    m, b = torch.randn(rank, H * d, generator=g) / rank ** 0.5, 3.0 + torch.randn(H * d, generator=g)
    low = 2 * H * d + H * dv + 2
    state = torch.full((5, H, d, dv), float("nan"), device="cuda:0")
    for s in slots:
        state[s].zero_()
    got = [[], []]
    for k, step in enumerate(recurrence_steps(lens, SIZES)):
        portions = [(slots[s], first, n) for s, first, n in step]
        rows = torch.cat([proj[s][first:first + n] for s, first, n in step] + ([torch.full((1, cols), 1e4).to(dtype)] if k % 2 else []))
        if k % 2:
            portions.append((slots[0], -1, 1))
        ctx = step_arrays(portions)
        o = R.linear_recurrence(rows.cuda(), 0, H * d, 2 * H * d, R.KEY_DECAY, H, d, dv, state, ctx.state_slot, ctx.q_start,
                                ctx.positions, gate_map=dev(m), gate_bias=dev(b), low_off=low, q_scale=0.3, power=1 / 5.0)
        at = 0
        for s, _, n in step:
            got[s].append(o[at:at + n].cpu().double())
            at += n
    for s, n in enumerate(lens):
        x = proj[s].double()
        alpha = torch.sigmoid(x[:, low:low + rank] @ m.double() + b.double()) ** (1 / 5.0)
        want, S = plain.gla_scan(0.3 * x[:, :H * d].view(n, H, d), x[:, H * d:2 * H * d].view(n, H, d),
                                 x[:, 2 * H * d:2 * H * d + H * dv].view(n, H, dv), alpha.view(n, H, d), torch.zeros(H, d, dv, dtype=plain.F))
        assert (torch.cat(got[s]).view(n, H, dv) - want).abs().max() < 3e-5 * want.abs().max()
        assert (state[slots[s]].cpu().double() - S).abs().max() < 3e-5 * S.abs().max()
    assert torch.isnan(state[[0, 2, 4]]).all()


@pytest.mark.parametrize("H,d,dv", DIMS + [(6, 64, 32), (4, 160, 20)])
@pytest.mark.parametrize("groups", [1, 2])
def test_recurrence_with_step_sizes(H, d, dv, groups):
    from dispec_b200.ops import recurrence as R
    if H % groups:
        groups = H
    g = torch.Generator().manual_seed(d + groups)
    lens, slots = [150, 90], [0, 2]
    cols = H * dv + 2 * groups * d
    rows = [torch.randn(n, cols, generator=g) for n in lens]
    dt = [torch.rand(n, H, generator=g) for n in lens]
    alog, D = torch.randn(H, generator=g) - 3.0, torch.randn(H, generator=g)
    state = torch.full((4, H, d, dv), float("nan"), device="cuda:0")
    for s in slots:
        state[s].zero_()
    got = [[], []]
    for k, step in enumerate(recurrence_steps(lens, SIZES)):
        portions = [(slots[s], first, n) for s, first, n in step]
        z = torch.cat([rows[s][first:first + n] for s, first, n in step] + ([torch.full((1, cols), 1e4)] if k % 2 else []))
        t = torch.cat([dt[s][first:first + n] for s, first, n in step] + ([torch.ones(1, H)] if k % 2 else []))
        if k % 2:
            portions.append((slots[1], -1, 1))
        steps = torch.stack([t, torch.exp(-torch.exp(alog) * t)], dim=1)
        ctx = step_arrays(portions)
        o = R.linear_recurrence(dev(z), H * dv + groups * d, H * dv, 0, R.STEP_DECAY, H, d, dv, state, ctx.state_slot, ctx.q_start,
                                ctx.positions, steps=dev(steps), skip=dev(D), num_groups=groups)
        at = 0
        for s, _, n in step:
            got[s].append(o[at:at + n].cpu().double())
            at += n
    for s, n in enumerate(lens):
        x = rows[s].double()
        B, C = (x[:, H * dv + i * groups * d:H * dv + (i + 1) * groups * d].view(n, groups, d).repeat_interleave(H // groups, dim=1) for i in (0, 1))
        want, S = plain.ssd_scan(x[:, :H * dv].view(n, H, dv), B, C, dt[s].double(), alog.double(), D.double(), torch.zeros(H, d, dv, dtype=plain.F))
        assert (torch.cat(got[s]).view(n, H, dv) - want).abs().max() < 3e-5 * want.abs().max()
        assert (state[slots[s]].cpu().double() - S).abs().max() < 3e-5 * S.abs().max()
    assert torch.isnan(state[[1, 3]]).all()


# ----------------------------------------------------------------------- a window with kept first keys
def scattered(lens, page, G, widths, g, dtype):
    """Random keys and values of requests of the given lengths in pools of scattered pages, NaN elsewhere."""
    n_pages = sum(-(-n // page) for n in lens) + 3
    perm = torch.randperm(n_pages, generator=g).tolist()
    width = max(-(-n // page) for n in lens)
    pools = [torch.full((n_pages, G, page, w), float("nan")) for w in widths]
    tables, rows = [], [[] for _ in widths]
    for n in lens:
        need = -(-n // page)
        tables.append([perm.pop() for _ in range(need)] + [-1] * (width - need))
        for i, w in enumerate(widths):
            r = torch.randn(n, G, w, generator=g).to(dtype).float()
            rows[i].append(r)
            for j in range(n):
                pools[i][tables[-1][j // page], :, j % page] = r[j]
    return tables, rows, pools


def give_back(tables, stored, page, window, keep):
    """Page ids the cache manager would have taken back become -1."""
    out = [list(t) for t in tables]
    for t, n in zip(out, stored):
        for p in range(-(-keep // page), max(0, n - window + 1) // page):
            t[p] = -1
    return out


@pytest.mark.parametrize("kernel", ["32-bit", "tensor cores"])
@pytest.mark.parametrize("H,G,dk,dv,page,window,keep", [(4, 2, 16, 32, 8, 21, 3), (8, 2, 64, 128, 16, 64, 70), (4, 4, 32, 16, 16, 100, 16),
                                                        (6, 1, 16, 16, 4, 5, 1), (2, 2, 32, 48, 32, 130, 200)])
def test_attention_kernels_see_the_window_and_the_kept_first_keys(kernel, H, G, dk, dv, page, window, keep):
    """Two single tokens (on tensor cores also with their keys cut into shares) and a portion of a prompt;
    every query is aimed at one key: the first of its window, the one before it, the last kept one, the one
    after it, position 0, its own position, the next one (stored, invisible), both sides of a page's edge."""
    from dispec_b200.ops import attention as AO
    from dispec_b200.ops import library
    dtype = torch.float32 if kernel == "32-bit" else torch.bfloat16
    g = torch.Generator().manual_seed(H * dk + window)
    lens, q_lens = [3 * page + window + keep, 431, window + keep + 190], [1, 1, 150]
    tables, (keys, vals), (k_pool, v_pool) = scattered(lens, page, G, (dk, dv), g, dtype)
    tables = give_back(tables, [n - q for n, q in zip(lens, q_lens)], page, window, keep)
    seq_of = [s for s, q in enumerate(q_lens) for _ in range(q)]
    pos = [n - q + i for n, q in zip(lens, q_lens) for i in range(q)]
    T = len(pos)
    scale = 0.31
    q = torch.randn(T, H, dk, generator=g) * 0.1
    star = []
    for t in range(T):
        p, n = pos[t], lens[seq_of[t]]
        first = max(0, p - window + 1)
        star.append([first, max(first - 1, 0), keep - 1, min(keep, p), 0, p, min(p + 1, n - 1), (first // page + 1) * page - 1,
                     min((first // page + 1) * page, p), min(keep // 2, p)][t % 10])
        for h in range(H):
            k = keys[seq_of[t]][star[t], h // (H // G)]
            q[t, h] += 14.0 / scale * k / k.norm() ** 2
    q = q.to(dtype).float()
    cache = SimpleNamespace(key_pool=dev(k_pool, dtype), value_pool=dev(v_pool, dtype), page_table=i32(tables))
    arrays = step_arrays([(0, n - ql, ql) for n, ql in zip(lens, q_lens)])
    qd = dev(q.reshape(T, H * dk), dtype)
    wide = torch.full((T, H * dv + 16), float("nan"), dtype=dtype, device="cuda:0")
    outs = []
    if kernel == "32-bit":
        out = wide[:, 8:8 + H * dv]
        AO.paged_attention_generic(qd, H * dk, cache.key_pool, cache.value_pool, cache.page_table, arrays.positions,
                                   arrays.seq_of_token, out, H, G, dk, window, scale, keep_first=keep)
        outs.append(out.float().cpu().double())
    else:
        tpt = AO.sink_tokens_per_tile(H // G, dk, dv)
        tiles = [(s, a) for s, ql in enumerate(q_lens) for a in range(0, ql, tpt)]
        for splits in (1, 2, 5, 16):
            wide.fill_(float("nan"))
            out = wide[:, 8:8 + H * dv]
            AO.sink_attention_tiles(qd, cache.key_pool, cache.value_pool, cache.page_table, arrays.q_start, i32(lens),
                                    i32([s for s, _ in tiles]), i32([a for _, a in tiles]), len(tiles), out, H, G, window, scale,
                                    False, num_single=2, splits=splits, keep_first=keep)
            outs.append(out.float().cpu().double())
    assert library.device_error() == 0  # no page that was given back was looked up
    assert torch.isnan(wide[:, :8].float()).all() and torch.isnan(wide[:, 8 + H * dv:].float()).all()
    stood_out = hidden = 0
    for t in range(T):
        s, p = seq_of[t], pos[t]
        args = (q[t:t + 1].double(), keys[s][:p + 1].double(), vals[s][:p + 1].double(), torch.tensor([p]), torch.arange(p + 1))
        want = plain.softmax_attention(*args, scale, window, keep)[0].reshape(-1)
        for out in outs:
            assert (out[t] - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.04) * max(1.0, want.abs().max().item()), (t, star[t], p)
        seen = star[t] <= p and (p - star[t] < window or star[t] < keep)
        ref = vals[s][star[t]].repeat_interleave(H // G, dim=0).double().reshape(-1)
        if seen:
            stood_out += (want - ref).abs().max() < 0.2
        else:
            hidden += (want - ref).abs().max() > 0.3
    assert stood_out > T // 3 and hidden > 0  # the aimed-at keys carry results, the invisible ones do not


# ----------------------------------------------------------------------- the joined mixers
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("left,right,scales", [
    (bu.left(4, 2, 16, 8, 4, window=20, keep=3, rot=8, bands=(3.0, 1.0, 3.0, 64)), bu.right(4, 16, 24, 2, 2, 4), (0.7, 1.4)),
    (bu.left(5, 5, 6, 10, 2, window=9, keep=11, rot=6), bu.right(3, 5, 7, 3, 5, 5), (-1.1, 0.9)),
    (bu.left(8, 2, 64, 32, 3, window=64, keep=4, rot=32), bu.right(8, 32, 64, 4, 4, 2), (1.0, 0.0)),
    (bu.left(2, 1, 8, 8, 1), bu.right(2, 8, 16, 1, 1, 1), (0.0, 1.0))])
def test_parallel_part_against_the_plain_mixers(left, right, scales, dtype):
    """The mixer alone: a long portion, single tokens, portions down to two tokens."""
    from dispec_b200.engine.batch import LayerCacheView, LayerStateView
    from dispec_b200.models.bepepel import BepepelConfig, _mixer_spec
    from dispec_b200.models.model import build_part
    g = torch.Generator().manual_seed(left["dim"] + right["state"])
    W, n, page = 48, 200, 8
    layer = bu.parallel(left, right, scales)
    cfg = BepepelConfig.from_dict(bu.model(W, 8, [layer], eps=1e-5))
    weights = {k: v for k, v in bu.random_weights(bu.model(W, 8, [layer]), 5).items() if ".mix." in k}
    bindings = []
    part = build_part(_mixer_spec(cfg, "parallel", layer["mixer"], "l0.mix."), {}, bindings)
    assert sorted(c for _, names in bindings for c, _ in names.values()) == sorted(weights)
    for p, names in bindings:
        p.load({local: dev(weights[c], dtype if spec.dtype == "model" else torch.float32) for local, (c, spec) in names.items()})
    for m in part.mixers:
        if hasattr(m, "position_encoding") and hasattr(m.position_encoding, "prepare"):
            m.position_encoding.prepare("cuda:0")
    part.prepare("cuda:0")
    x = torch.randn(n, W, generator=g).bfloat16().float()
    want, _ = plain.parallel(x.double(), {k: v.double() for k, v in weights.items()}, "l0.mix.", layer["mixer"], 1e-5, torch.arange(n))
    n_pages = n // page + 2
    table = i32([torch.randperm(n_pages, generator=g).tolist()[:n // page]])
    G = left["kv_heads"]
    pools = {"key": torch.full((n_pages, G, page, left["dim"]), float("nan"), dtype=dtype, device="cuda:0"),
             "value": torch.full((n_pages, G, page, left["vdim"]), float("nan"), dtype=dtype, device="cuda:0")}
    need = part.cache_need()
    cache = LayerCacheView(pools, table, 0, True, page, n_pages, need.window)
    buffers = [torch.zeros((3,) + tuple(s.shape), device="cuda:0") for s in part.state_need()]
    tiles_of = [t for t in (part.tokens_per_attention_tile() or ()) if t]
    got, start = [], 0
    for stop in (120, 121, 122, 160, 162, 199, 200):
        ql = stop - start
        ctx = step_arrays([(2, start, ql)])
        ctx.dtype, ctx.ctx_len, ctx.max_ctx_len, ctx.num_decode_seqs = dtype, i32([stop]), stop, 1 if ql == 1 else 0
        ctx.attention_tiles = {t: (i32([0] * len(range(0, ql, t))), i32(list(range(0, ql, t))), len(range(0, ql, t))) for t in tiles_of}
        state = tuple(LayerStateView(b, ctx.state_slot) for b in buffers)
        got.append(part.forward(ctx, dev(x[start:stop], dtype), cache, state).cpu().double())
        start = stop
    assert (torch.cat(got) - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.04) * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,d,dv,rank,tau", [(4, 16, 8, 16, 8.0), (3, 6, 10, 5, 1.0), (2, 128, 96, 24, 16.0)])
def test_gated_linear_attention_part_against_the_plain_mixer(H, d, dv, rank, tau, dtype):
    from dispec_b200.engine.batch import LayerStateView
    from dispec_b200.parts.linear_attention import GatedLinearAttention
    g = torch.Generator().manual_seed(d)
    W, n = 48, 130
    layer = bu.gla(H, d, dv, tau)
    P = {k[7:]: v for k, v in bu.random_weights(bu.model(W, 8, [layer]), 6, rank).items() if ".mix." in k}
    part = GatedLinearAttention(W, H, d, dv, rank, tau, 1e-5)
    part.load({("a2.bias" if k == "a2.b" else k + ".weight"): dev(v, dtype if k in ("q", "k", "v", "g", "o", "a1") else torch.float32)
               for k, v in P.items()})
    x = torch.randn(n, W, generator=g).bfloat16().float()
    want, _ = plain.gla(x.double(), {"m." + k: v.double() for k, v in P.items()}, "m.", layer["mixer"], 1e-5, torch.arange(n))
    buf = torch.zeros(2, H, d, dv, device="cuda:0")
    got, start = [], 0
    for stop in (70, 71, 72, 110, 112, 130):
        ctx = step_arrays([(1, start, stop - start)])
        got.append(part.forward(ctx, dev(x[start:stop], dtype), None, LayerStateView(buf, ctx.state_slot)).cpu().double())
        start = stop
    assert (torch.cat(got) - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.05) * max(1.0, want.abs().max().item())
    assert math.isfinite(float(buf[1].abs().max())) and float(buf[0].abs().max()) == 0.0
