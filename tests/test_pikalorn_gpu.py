"""Pikalorn through the engine against the plain implementation.

Replays through bin/trace_run: the same requests whole, with their last tokens one by one, in
portions of changing size down to two tokens, and mixed (up to four live, portions beside single
tokens, few pages and four state slots so that both are used again, freed pages filled with NaN),
in float32 and bfloat16, also from captured CUDA graphs.  "Sharp" variants scale the scores and
lengthen the memories so that a lost far key, a sink left out or a lost state shows.  The stream after
every layer.  Generation through LLMEngine, ContinuousBatchingEngine and the command line.  The
kernels and parts one by one."""
import math
from types import SimpleNamespace

import pytest
import torch

import pikalorn_util as pu
import plain_pikalorn as plain
import replay_util as ru

pytestmark = pytest.mark.gpu

LENGTHS = {"mix": [1, 9, 40, 131, 260], "odd": [2, 17, 64, 150], "wide": [3, 33, 97, 230], "long": [4, 299, 705]}


def rounded_inputs(config, weights, ids, monkeypatch):
    """The plain logits when every sublayer's input is rounded to bfloat16: how far one rounding alone moves
    each position (a head divided by a small root mean square or length magnifies it)."""
    exact = plain.rms
    with monkeypatch.context() as m:
        m.setattr(plain, "rms", lambda *a: exact(*a).bfloat16().double())
        return plain.forward(config, weights, ids)[0].float()


def replay(name, dtype, tmp_path, monkeypatch, cuda_graph=False, sharp=False):
    spec = pu.CONFIGS[name]
    model_dir = str(tmp_path / "model")
    config, weights = pu.make_folder(model_dir, name, sharp=sharp)
    prompts = {f"p{n}": ru.random_ids(n, config["vocab"], 100 + n) for n in LENGTHS[name]}
    trace, peak = ru.build_four_mode_trace(prompts, spec["page_size"])
    got = ru.run_trace(model_dir, dtype, trace, peak, str(tmp_path / "out"), page_size=spec["page_size"],
                       cuda_graph=cuda_graph, max_requests=4)
    refs = {n: plain.forward(config, weights, ids)[0].float() for n, ids in prompts.items()}
    moved = {n: (rounded_inputs(config, weights, ids, monkeypatch) - refs[n]).abs().amax(-1) if dtype == "bfloat16" else None
             for n, ids in prompts.items()}
    modes = set()
    for (step, rid, pos), row in got.items():
        mode, pname = rid.split("/")
        modes.add(mode.rstrip("01"))
        assert torch.isfinite(row).all(), (step, rid, pos)
        err = (row - refs[pname][pos]).abs().max().item()
        scale = max(refs[pname][pos].abs().max().item(), 1e-3)
        bound = (1e-3 if sharp else 1e-4) * max(scale, 1.0) if dtype == "float32" \
            else 0.04 * scale + 0.02 + 3.0 * float(moved[pname][pos])
        assert err <= bound, f"first wrong place: step {step} request {rid} position {pos}: {err} (scale {scale})"
    assert modes == {"whole", "tail", "portions", "mixed"}


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "long"])
def test_replay_float32(name, tmp_path, monkeypatch):
    replay(name, "float32", tmp_path, monkeypatch)


@pytest.mark.parametrize("name", ["mix", "odd", "wide", "long"])
def test_replay_bfloat16(name, tmp_path, monkeypatch):
    replay(name, "bfloat16", tmp_path, monkeypatch)


@pytest.mark.parametrize("name", ["mix", "wide"])
def test_replay_bfloat16_single_token_steps_from_captured_graphs(name, tmp_path, monkeypatch):
    replay(name, "bfloat16", tmp_path, monkeypatch, cuda_graph=True)


@pytest.mark.parametrize("name", ["mix", "odd", "long"])
def test_replay_float32_sharp_keys_and_long_memories(name, tmp_path, monkeypatch):
    replay(name, "float32", tmp_path, monkeypatch, sharp=True)


# ------------------------------------------------------------------ the stream after every layer
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name in ("mix", "odd", "wide"):
        d = str(tmp_path_factory.mktemp(f"pikalorn_{name}"))
        out[name] = (d,) + pu.make_folder(d, name)
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
    r = ModelRunner(model, page_size=pu.CONFIGS[name]["page_size"], num_pages=16, max_num_seqs=2)
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
    folder, config, weights = folders["mix"]
    engine = LLMEngine(load(folder, dtype), num_blocks=32, cuda_graph=dtype == "bfloat16")
    for n in (1, 9, 40):  # the same engine: pages and slots are used again
        prompt = ru.random_ids(n, config["vocab"], 300 + n)
        got = engine.generate(prompt, 10, SamplingParams(temperature=0.0))
        assert len(got) == 10
        assert_greedy(weights, config, prompt, got, dtype)
    cache = engine.runner.cache
    assert all(cache.num_free_pages(g) == 32 for g in range(len(cache.groups)))


def test_long_decoding_float32(folders):
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
    folder, config, weights = folders["wide"]
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
    """`python -m dispec_b200 generate` on a Pikalorn folder: greedy tokens equal the plain ones; `random` writes a
    folder for the same configuration that `generate` serves too."""
    import json
    import os
    import subprocess
    import sys
    folder = str(tmp_path / "model")
    config, weights = pu.make_folder(folder, "odd")
    env = dict(os.environ, PYTHONPATH=ru.ROOT)
    prompts = [[5, 17, 3, 90], list(range(7, 33))]
    cmd = [sys.executable, "-m", "dispec_b200", "generate", "--dtype", "float32", "--max-new", "8", "--block-size", "8",
           "--num-blocks", "48", "--max-batch-tokens", "16", "--chunk-size", "6"]
    for p in prompts:
        cmd += ["--prompt-ids", ",".join(map(str, p))]
    cfg_path = tmp_path / "config.json"
    cfg_path.write_text(json.dumps(config))
    made = str(tmp_path / "made")
    subprocess.run([sys.executable, "-m", "dispec_b200", "random", "--config", str(cfg_path), "--out", made, "--seed", "5",
                    "--std", "0.08"], check=True, env=env, cwd=ru.ROOT)
    from safetensors.torch import load_file
    made_weights = {k: v.float() for k, v in load_file(os.path.join(made, "model.safetensors")).items()}
    assert {k: tuple(v.shape) for k, v in made_weights.items()} == plain.tensor_shapes(config)
    for where, w in ((folder, weights), (made, made_weights)):
        proc = subprocess.run(cmd + ["--model", where], check=True, env=env, cwd=ru.ROOT, capture_output=True, text=True)
        lines = [json.loads(ln) for ln in proc.stdout.splitlines() if ln.startswith("{")]
        assert [ln["prompt_tokens"] for ln in lines] == [len(p) for p in prompts]
        for ln, prompt in zip(lines, prompts):
            assert len(ln["output_ids"]) == 8
            assert_greedy(w, config, prompt, ln["output_ids"], "float32")


# ----------------------------------------------------------------------- kernels and parts one by one
def dev(t, dtype=torch.float32):
    return t.to(device="cuda:0", dtype=dtype).contiguous()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda:0")


def step_arrays(portions, tiles=(8,)):
    """``portions``: (slot, first position, tokens) of each request, single tokens first -> the step's arrays, with
    lists of tiles of the given sizes.  A first position of -1 makes a padding row."""
    pos, seq, start, ctx_len = [], [], [0], []
    for s, (_, first, n) in enumerate(portions):
        pos += [-1] * n if first < 0 else list(range(first, first + n))
        seq += [s] * n
        start.append(start[-1] + n)
        ctx_len.append(0 if first < 0 else first + n)
    singles = [p[2] == 1 for p in portions]
    n_dec = singles.index(False) if False in singles else len(singles)
    assert not any(singles[n_dec:])
    lists = {}
    for size in tiles:
        at = [(s, a) for s, p in enumerate(portions) for a in range(0, p[2], size)]
        lists[size] = (i32([s for s, _ in at]), i32([a for _, a in at]), len(at))
    return SimpleNamespace(positions=i32(pos), seq_of_token=i32(seq), q_start=i32(start), ctx_len=i32(ctx_len),
                           state_slot=i32([p[0] for p in portions]), attention_tiles=lists, num_decode_seqs=n_dec,
                           max_ctx_len=max(ctx_len))


# steps of three requests (slot 4, 1 and 2), in portions; single tokens are put first by `walk`
STEPS = [(2, 1, 9), (1, 1, 1), (3, 17, 1), (1, 5, 8), (40, 2, 24), (60, 60, 60)]


def walk(lens, steps, run):
    """Runs the requests of ``lens`` (slot -> tokens) in the given portions beside padding rows:
    ``run(ctx, [(slot, first, n)])`` for every step."""
    done = {s: 0 for s in lens}
    for k, step in enumerate(steps):
        portions = []
        for s, n in zip(lens, step):
            n = min(n, lens[s] - done[s])
            if n:
                portions.append((s, done[s], n))
                done[s] += n
        if k % 2:  # a padding row names a slot that belongs to someone else
            portions.append((list(lens)[0], -1, 1))
        portions.sort(key=lambda p: p[2] != 1)
        if portions:
            run(step_arrays(portions), portions)
    assert done == lens


@pytest.mark.parametrize("kind", ["plain", "forgetful", "same_keys"])
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 16, 24), (3, 1, 5, 7), (2, 2, 64, 40), (4, 1, 128, 96), (1, 1, 33, 20), (2, 2, 200, 17),
                                          (2, 1, 300, 9)])
def test_delta_rule_kernels_carry_the_state_from_portion_to_portion(H, G, dim, vdim, kind):
    """Portions shorter and longer than a run beside single tokens and padding rows; slots of others filled with NaN.
    "forgetful": decays down to exp(-200); "same_keys": every key is one of two opposite ones, written at nearly full
    strength without decay, where each write undoes most of what the state holds."""
    from dispec_b200.ops import recurrence as RO
    g = torch.Generator().manual_seed(H * dim + vdim)
    lens = {4: 71, 1: 66, 2: 55}
    rows, steps, state0 = {}, {}, {}
    for s, n in lens.items():
        q, k = (torch.nn.functional.normalize(torch.randn(n, G, dim, generator=g), dim=-1) for _ in range(2))
        beta, lg = torch.rand(n, H, generator=g), -torch.rand(n, H, generator=g) * 0.2
        if kind == "forgetful":
            lg = lg * 10.0 ** (torch.rand(n, H, generator=g) * 5 - 2)
        if kind == "same_keys":
            k = k[:1] * torch.where(torch.rand(n, G, 1, generator=g) < 0.5, -1.0, 1.0)
            beta, lg = 0.9 + 0.1 * beta, lg * 0.0
        rows[s] = torch.cat([(q * dim ** -0.5).reshape(n, -1), k.reshape(n, -1), torch.randn(n, H * vdim, generator=g)], 1)
        steps[s] = torch.stack([beta, lg], 1)
        state0[s] = torch.randn(H, dim, vdim, generator=g)
    state = torch.full((6, H, dim, vdim), float("nan"), device="cuda:0")
    for s in lens:
        state[s] = dev(state0[s])
    got = {s: [] for s in lens}

    def run(ctx, portions):
        r = torch.cat([rows[s][a:a + n] if a >= 0 else torch.full((1, rows[s].shape[1]), 1e6) for s, a, n in portions])
        st = torch.cat([steps[s][a:a + n] if a >= 0 else torch.ones(1, 2, H) for s, a, n in portions])
        wide = torch.full((r.shape[0], (r.shape[1] + 7) // 4 * 4), float("nan"), device="cuda:0")
        wide[:, :r.shape[1]] = dev(r)
        out = RO.delta_rule(ctx, wide[:, :r.shape[1]], dev(st), H, G, dim, vdim, state)
        at = 0
        for s, a, n in portions:
            if a >= 0:
                got[s].append(out[at:at + n].cpu().double())
            at += n

    walk(lens, STEPS, run)
    for s, n in lens.items():
        q, k, v = rows[s].double().split([G * dim, G * dim, H * vdim], 1)
        pick = lambda x: x.view(n, G, dim).repeat_interleave(H // G, dim=1)
        want, S = plain.delta_scan(pick(q), pick(k), v.view(n, H, vdim), steps[s][:, 0].double(), torch.exp(steps[s][:, 1].double()), state0[s].double())
        o = torch.cat(got[s]).view(n, H, vdim)
        assert (o - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item()), kind
        assert (state[s].cpu().double() - S).abs().max() < 2e-5 * max(1.0, S.abs().max().item())
    assert torch.isnan(state[[0, 3, 5]]).all()


@pytest.mark.parametrize("taps,G,dim,H,vdim", [(1, 2, 6, 4, 10), (2, 1, 37, 3, 5), (4, 3, 128, 3, 64), (4, 2, 300, 2, 16), (5, 2, 8, 2, 200), (9, 1, 4, 1, 4)])
def test_conv_heads_kernel_carries_its_inputs_from_portion_to_portion(taps, G, dim, H, vdim):
    from dispec_b200.ops import short_conv as SC
    g = torch.Generator().manual_seed(taps * dim)
    channels = 2 * G * dim + H * vdim
    cols = (channels + 2 * H + 10) // 4 * 4
    w, dtb, alog = torch.randn(channels, taps, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g)
    lens = {4: 71, 1: 66, 2: 55}
    u = {s: torch.randn(n, cols, generator=g) for s, n in lens.items()}
    u[4][7, channels + H] = 60.0  # a softplus far in its linear part
    u[1][20:23, :dim] = 0.0  # a head of zeros (or nearly: its length is what the small number inside the root makes it)
    hist = torch.full((6, taps - 1, channels), float("nan"), device="cuda:0")
    for s in lens:
        hist[s].zero_()
    got = {s: ([], []) for s in lens}

    def run(ctx, portions):
        rows = torch.cat([u[s][a:a + n] if a >= 0 else torch.full((1, cols), 1e6) for s, a, n in portions])
        out, steps = SC.conv_heads(dev(rows), dev(w.t()), hist if taps > 1 else None, ctx, G, G, dim, H, vdim, 1e-6, 0.3, channels,
                                   channels + H, dev(dtb), dev(alog))
        at = 0
        for s, a, n in portions:
            if a >= 0:
                got[s][0].append(out[at:at + n].cpu().double())
                got[s][1].append(steps[at:at + n].cpu().double())
            at += n

    walk(lens, STEPS, run)
    for s, n in lens.items():
        y, kept = plain.short_conv(u[s][:, :channels].double(), w.double(), torch.zeros(taps - 1, channels, dtype=plain.F))
        q, k, v = plain.silu(y).split([G * dim, G * dim, H * vdim], 1)
        want = torch.cat([plain.unit(q.reshape(n, G, dim)).reshape(n, -1) * 0.3, plain.unit(k.reshape(n, G, dim)).reshape(n, -1), v], 1)
        assert (torch.cat(got[s][0]) - want).abs().max() < 2e-5 * max(1.0, want.abs().max().item())
        if taps > 1:
            assert (hist[s].cpu().double() - kept).abs().max() < 1e-6
        steps, x = torch.cat(got[s][1]), u[s].double()
        assert (steps[:, 0] - torch.sigmoid(x[:, channels:channels + H])).abs().max() < 1e-6
        lg = -torch.exp(alog.double()) * plain.softplus(x[:, channels + H:channels + 2 * H] + dtb.double())
        assert ((steps[:, 1] - lg).abs() / (1 + lg.abs())).max() < 1e-5
    if taps > 1:
        assert torch.isnan(hist[[0, 3, 5]]).all()


# ----------------------------------------------------------------------- attention with sinks
def scattered(lens, page, widths, heads, g, dtype):
    """Rows of random values for requests of the given lengths in pools of scattered pages (NaN everywhere else):
    (page tables, per width the requests' rows [n, heads, width], per width the pool)."""
    n_pages = sum(-(-n // page) for n in lens) + 3
    perm = torch.randperm(n_pages, generator=g).tolist()
    width = max(-(-n // page) for n in lens)
    pools = [torch.full((n_pages, heads, page, w), float("nan")) for w in widths]
    tables, rows = [], [[] for _ in widths]
    for n in lens:
        need = -(-n // page)
        tables.append([perm.pop() for _ in range(need)] + [-1] * (width - need))
        for i, w in enumerate(widths):
            r = torch.randn(n, heads, w, generator=g).to(dtype).float()
            rows[i].append(r)
            for j in range(n):
                pools[i][tables[-1][j // page], :, j % page] = r[j]
    return tables, rows, [dev(p, dtype) for p in pools]


def aims(p, n, page):
    """Keys a query at position p of n tokens is aimed at in turn: the sequence's first tokens, both sides of a page
    border, its own position, the next one (stored, invisible), a far one."""
    return [0, 1, page - 1, page, p, min(p + 1, n - 1), p // 2]


@pytest.mark.parametrize("tensor_cores", [False, True])
@pytest.mark.parametrize("H,R,r,page,sink", [(4, 80, 16, 8, 0.0), (10, 16, 16, 16, 3.0), (6, 112, 32, 16, -2.0), (2, 320, 32, 32, 1.0),
                                             (66, 192, 64, 16, 2.0), (3, 400, 16, 16, 30.0), (5, 20, 6, 4, 1.0)])
def test_latent_attention_with_a_sink_and_interleaved_turns(H, R, r, page, sink, tensor_cores):
    from dispec_b200.ops import latent as LO
    from dispec_b200.ops import library
    if tensor_cores and (R % 16 or r % 16):
        pytest.skip("sizes of the 32-bit kernel")
    g = torch.Generator().manual_seed(H + R)
    lens, q_lens, dtype = [3 * page + 5, 700, 9 * page + 50], [1, 1, 45], torch.bfloat16 if tensor_cores else torch.float32
    tables, (lat, rk), (c_pool, r_pool) = scattered(lens, page, [R, r], 1, g, dtype)
    z = torch.randn(H, generator=g) + sink
    rot = {"dims": r, "base": 50.0, "scaling": {"factor": 3.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    freq, mag = plain.frequencies(rot)
    portions = [(s, n - ql, ql) for s, (n, ql) in enumerate(zip(lens, q_lens))]
    tpt = LO.mma_tokens_per_tile(H)
    ctx = step_arrays(portions, tiles=(tpt,))
    pos, seq = ctx.positions.tolist(), ctx.seq_of_token.tolist()
    T = len(pos)
    qa, q_rot = torch.randn(T, H, R, generator=g) * 0.05, torch.randn(T, H, r, generator=g) * 0.05
    star = [aims(pos[t], lens[seq[t]], page)[t % 7] for t in range(T)]
    for t in range(T):
        if t % 3:  # every third query is aimed at nothing: there the sink has its share
            c = lat[seq[t]][star[t], 0]
            qa[t] += 8.0 * c / c.norm() ** 2 * math.sqrt(R)
    qraw = torch.cat([torch.zeros(T, H, 8), q_rot], -1).reshape(T, -1)
    qraw = qraw.to(dtype)
    scale, table = 0.21, i32(tables)
    common = (dev(qa.reshape(T, -1)), dev(qraw, dtype), 8 + r, 8, dev(freq.float()), r, c_pool, r_pool, table)
    if tensor_cores:
        assert LO.mma_supported(R, r, dtype)
        out = LO.latent_attention_tiles(ctx, *common, H, scale, layout="interleaved", magnitude=mag, sink=dev(z))
    else:
        out = LO.latent_attention(*common, ctx.positions, ctx.seq_of_token, H, scale, torch.float32, layout="interleaved",
                                  magnitude=mag, sink=dev(z))
    assert library.device_error() == 0
    out = out.float().cpu().double().view(T, H, R)
    for t in range(T):
        s, p = seq[t], torch.tensor([pos[t]])
        q = torch.cat([qa[t].double(), plain.turn(qraw.double().view(T, H, -1)[t:t + 1, :, 8:], p, rot, True)[0]], -1)[None]
        k = torch.cat([lat[s][:, 0], rk[s][:, 0]], -1).double()[:, None].expand(-1, H, -1)
        v = lat[s].double().expand(-1, H, -1)
        want = plain.sink_softmax_attention(q, k, v, p, torch.arange(lens[s]), scale, z.double())[0]
        tol = 0.03 if tensor_cores else 2e-4
        assert (out[t] - want).abs().max() < tol * max(1.0, want.abs().max().item()), (t, star[t])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,rot,page,group_scale", [(4, 2, 16, 8, 8, 1.0), (5, 1, 10, 2, 4, 3.0), (8, 1, 64, 64, 16, 1.0), (6, 3, 128, 32, 32, 4.0),
                                                        (4, 4, 6, 0, 8, 1.0), (12, 1, 48, 48, 16, 2.0)])
def test_attention_part_whose_values_are_its_keys(H, G, d, rot, page, group_scale, dtype):
    """The whole mixer (biases, head norms, rotation, raw keys as values, sinks, output gate) over portions of three
    requests in scattered pages, against the plain mixer on the same rows."""
    from dispec_b200.ops import attention as AO
    from dispec_b200.parts.attention import SinkAttention
    from dispec_b200.parts.rotary import NoPositionEncoding, RotaryEncoding
    g = torch.Generator().manual_seed(H * d)
    W, m = 48, {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": group_scale * d ** -0.5, "rot": {"dims": rot, "base": 300.0}}
    shapes = {"q": (H * d, W), "k": (G * d, W), "g": (H * d, W), "o": (W, H * d), "q.b": (H * d,), "k.b": (G * d,), "o.b": (W,),
              "q.norm": (d,), "k.norm": (d,), "sink": (H,)}
    P = {n: (torch.randn(s, generator=g) / (s[-1] ** 0.5 if len(s) == 2 else 1.0)).bfloat16().float() for n, s in shapes.items()}
    enc = RotaryEncoding(d, 300.0, rot, exact_table=True) if rot else NoPositionEncoding()
    if rot:
        enc.prepare("cuda:0")
    part = SinkAttention(W, H, G, d, d, m["scale"], enc, sink="learned", head_norm=True, norm_eps=1e-5, bias=True, values="keys", out_gate=True)
    wide = {"q": "q.weight", "k": "k.weight", "g": "g.weight", "o": "o.weight", "q.b": "q.bias", "k.b": "k.bias", "o.b": "o.bias"}
    small = {"q.norm": "q.norm.weight", "k.norm": "k.norm.weight", "sink": "sink"}
    part.load({**{l: dev(P[n], dtype) for n, l in wide.items()}, **{l: dev(P[n]) for n, l in small.items()}})
    assert part.cache_need().tensors[1].width == d
    lens = {4: 71, 1: 66, 2: 55}
    tables = {s: [10 * i + j for j in torch.randperm(9 if page > 4 else 20, generator=g).tolist()] for i, s in enumerate(lens)}
    if page == 4:
        tables = {s: [20 * i + j % 20 for j in t] for i, (s, t) in enumerate(tables.items())}
    h = {s: torch.randn(n, W, generator=g).bfloat16().float() for s, n in lens.items()}
    pools = [torch.full((60, G, page, d), float("nan"), dtype=dtype, device="cuda:0") for _ in range(2)]
    tpt = AO.sink_tokens_per_tile(H // G, d, d)
    got = {s: [] for s in lens}

    def run(ctx, portions):
        again = step_arrays(portions, tiles=(tpt,) if tpt else (8,))
        again.dtype = dtype
        rows = torch.cat([h[s][a:a + n] if a >= 0 else torch.full((1, W), 1e3) for s, a, n in portions])
        cache = SimpleNamespace(key_pool=pools[0], value_pool=pools[1], page_table=i32([tables[s] for s, _, _ in portions]), write=True)
        y = part.forward(again, dev(rows, dtype), cache, None)
        at = 0
        for s, a, n in portions:
            if a >= 0:
                got[s].append(y[at:at + n].cpu().double())
            at += n

    walk(lens, STEPS, run)
    for s, n in lens.items():
        want, _ = plain.attention(h[s].double(), {k: v.double() for k, v in P.items()}, "", m, 1e-5, torch.arange(n), None)
        tol = 1e-4 if dtype == torch.float32 else 0.04
        assert (torch.cat(got[s]) - want).abs().max() < tol * max(1.0, want.abs().max().item())


# ----------------------------------------------------------------------- the block
@pytest.mark.parametrize("dtype,W,ff,inner", [(torch.float32, 52, 30, 20), (torch.bfloat16, 64, 96, 40), (torch.bfloat16, 64, 96, 36),
                                              (torch.bfloat16, 256, 512, 384), (torch.bfloat16, 128, 40, 64), (torch.bfloat16, 60, 64, 64)])
@pytest.mark.parametrize("T", [1, 9, 150])
@pytest.mark.parametrize("with_ff", [True, False])
def test_parallel_block_joins_the_two_output_products(dtype, W, ff, inner, T, with_ff):
    """A stand-in mixer (its rows through tanh, an output bias) beside the gated unit, joined where the sizes allow."""
    from dispec_b200.parts.base import JoinableMixer, WideStream
    from dispec_b200.parts.block import ParallelPreNormBlock
    from dispec_b200.parts.norms import RMSNorm32
    from dispec_b200.parts.swiglu import SwiGLUFeedForward
    g = torch.Generator().manual_seed(W + inner)
    mat = lambda *s: (torch.randn(s, generator=g) / s[-1] ** 0.5).bfloat16().float()
    P = {"in": mat(inner, W), "o": mat(W, inner), "o.b": mat(W), "gate": mat(ff, W), "up": mat(ff, W), "down": mat(W, ff),
         "n": 1 + 0.2 * mat(W), "next": 1 + 0.2 * mat(W)}

    class Toy(JoinableMixer):
        def heads(self, ctx, z, cache, state, out):
            out.copy_(torch.tanh(z))

    toy = Toy()
    toy.out_columns, toy.w_in, toy.w_o, toy.b_o = inner, dev(P["in"], dtype), dev(P["o"], dtype), dev(P["o.b"], dtype)
    unit = SwiGLUFeedForward(W, ff, out_float32=True)
    unit.load({n + "_proj.weight": dev(P[n], dtype) for n in ("gate", "up", "down")})
    norms = []
    for n in ("n", "next"):
        norms.append(RMSNorm32(W, 1e-5))
        norms[-1].load({"weight": dev(P[n])})
    block = ParallelPreNormBlock(W, norms[0], toy, unit if with_ff else None)
    block.prepare("cuda:0")
    assert (block.w_joined is not None) == (with_ff and dtype == torch.bfloat16 and W % 8 == 0 and ff % 16 == 0 and inner % 8 == 0)
    x = 3 * torch.randn(T, W, generator=g)
    s, ctx = WideStream(dev(x), None), SimpleNamespace(dtype=dtype)
    out, nxt = block.forward(ctx, s, None, None, None, then_norm=(norms[1].weight, 1e-5))
    D = {k: v.double() for k, v in P.items()}
    h = plain.rms(x.double(), 1e-5, D["n"]).to(dtype).double()
    want = x.double() + torch.tanh(h @ D["in"].T) @ D["o"].T + D["o.b"] + (plain.feed_forward(h, D, "") if with_ff else 0.0)
    tol = 1e-4 if dtype == torch.float32 else 0.03
    assert out is s and (s.full.cpu().double() - want).abs().max() < tol * max(1.0, want.abs().max().item())
    want = plain.rms(s.full.cpu().double(), 1e-5, D["next"])
    assert nxt.dtype == dtype and (nxt.cpu().double() - want).abs().max() < (1e-5 if dtype == torch.float32 else 0.01) * want.abs().max()
    assert block.forward(ctx, s, nxt, None, None)[1] is None  # the last block keeps nothing pending
