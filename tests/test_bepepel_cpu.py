"""Bepepel without a GPU: the configuration reader, the builder's tensor list against the one the
tests derive on their own, ranks taken from the checkpoint, cache groups with kept first pages and
states, the table of banded frequencies, and the plain implementation against itself (token by token
and in portions through what it carries, against whole prompts; masks; a query aimed at one key)."""
import copy
import math

import pytest
import torch

import bepepel_util as bu
import plain_bepepel as plain
import replay_util as ru


class Shapes:
    """A checkpoint's names and shapes without its data."""

    def __init__(self, shapes):
        self._s = shapes

    def names(self):
        return list(self._s)

    def shape(self, name):
        return self._s[name]


def build(config, rank=16):
    from dispec_b200.config.model_config import load_model_config
    from dispec_b200.weights.loader import build_model
    cfg = load_model_config(copy.deepcopy(config)).with_tensor_shapes(Shapes(plain.tensor_shapes(config, rank)))
    return cfg, build_model(cfg)


@pytest.mark.parametrize("name", sorted(bu.CONFIGS))
def test_builder_asks_for_exactly_the_checkpoint_tensors(name):
    from dispec_b200.config.model_config import load_model_config
    config, rank = bu.CONFIGS[name]["config"], bu.CONFIGS[name]["rank"]
    cfg, m = build(config, rank)
    assert load_model_config(cfg.to_dict()) == cfg
    req, want = m.tensor_requirements(), plain.tensor_shapes(config, rank)
    assert set(req) == set(want)
    for n, spec in req.items():
        assert tuple(spec.shape) == tuple(want[n]), n
    assert [c.layer for c in m.schedule] == list(range(len(config["layers"])))


def test_ranks_follow_the_checkpoint_layer_by_layer():
    from dispec_b200.config.model_config import load_model_config
    from dispec_b200.weights.loader import WeightError, build_model, check_source
    config = copy.deepcopy(bu.CONFIGS["mix"]["config"])
    shapes = plain.tensor_shapes(config, [0, 3, 20, 0])
    cfg = load_model_config(config).with_tensor_shapes(Shapes(shapes))
    req = build_model(cfg).tensor_requirements()
    assert {n: tuple(s.shape) for n, s in req.items()} == shapes
    # without a checkpoint: the file's own rank, or 16
    config["layers"][1]["mixer"]["rank"] = 5
    req = build_model(load_model_config(config)).tensor_requirements()
    assert tuple(req["l1.mix.a1"].shape) == (5, 64) and tuple(req["l2.mix.a2"].shape) == (48, 16)

    class Broken(Shapes):
        def dtype(self, name):
            return torch.float32

    shapes["l1.mix.a2"] = (64, 4)  # does not fit a1
    with pytest.raises(WeightError, match="l1.mix.a2"):
        check_source(build_model(cfg), Broken(shapes), "here")


def test_caches_and_states_of_the_mixers():
    _, m = build(bu.CONFIGS["mix"]["config"])
    got = sorted((g.window, g.keep_first, [(t.name, t.num_heads, t.width) for t in g.tensors], g.num_slots) for g in m.cache_groups)
    assert got == [(0, 0, [("key", 1, 8), ("value", 1, 12)], 1), (20, 3, [("key", 2, 16), ("value", 2, 8)], 1)]
    # a parallel layer's left convolution, right matrix and right convolution; nothing is kept for single taps
    assert m.call_state == [(0, 1, 2), 3, 4, (5,)]
    assert [s.shape for s in m.state_needs] == [(3, 4 * 16 + 2 * 16 + 2 * 8), (4, 24, 16), (1, 64 + 2 * 2 * 24), (4, 16, 8),
                                                (2, 24, 20), (2, 16, 24)]
    assert all(s.dtype == "float32" for s in m.state_needs)


def test_the_norm_of_a_missing_feed_forward_may_be_present():
    _, m = build(bu.CONFIGS["mix"]["config"])  # its third layer has no feed-forward
    assert m.spec.optional_tensors == {"l2.norm2", "l2.norm2.b"}


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("low"), "low"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=7), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][1]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][1]["mlp"].update(kind="conv"), "not implemented"),
    (lambda c: c["layers"][1]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("ff"), "ff"),
    (lambda c: c.pop("width"), "width"),
])
def test_configuration_errors_name_the_key(change, word):
    from dispec_b200.config.model_config import ConfigError, load_model_config
    c = copy.deepcopy(bu.CONFIGS["mix"]["config"])
    change(c)
    with pytest.raises(ConfigError) as e:
        load_model_config(c)
    assert word in str(e.value)


def test_part_constructors_refuse_what_cannot_run():
    from dispec_b200.parts.attention import ConvAttention, SinkAttention
    from dispec_b200.parts.linear_attention import GatedLinearAttention
    from dispec_b200.parts.parallel import ParallelMixer
    from dispec_b200.parts.rotary import RotaryEncoding
    from dispec_b200.parts.state_space import StateSpaceDual
    from dispec_b200.parts.swiglu import SwiGLUFeedForward
    with pytest.raises(ValueError):
        ConvAttention(16, 4, 3, 8, 8, 0.5, None)
    with pytest.raises(ValueError):
        ConvAttention(16, 4, 2, 8, 8, 0.5, None, window=-1)
    with pytest.raises(ValueError):
        GatedLinearAttention(16, 2, 8, 8, 0, 4.0, 1e-6)
    with pytest.raises(ValueError):
        StateSpaceDual(16, 4, 8, 8, 3, 2, 1, 1e-6)
    with pytest.raises(ValueError):
        SwiGLUFeedForward(16, 8, act="tanh")
    with pytest.raises(ValueError):
        RotaryEncoding(16, 10000.0, banded=(4.0, 2.0, 1.0, 64))
    a = ConvAttention(16, 4, 2, 8, 8, 0.5, None)
    with pytest.raises(ValueError):  # two mixers with a paged cache
        ParallelMixer(a, ConvAttention(16, 4, 2, 8, 8, 0.5, None))
    with pytest.raises(ValueError):  # a mixer that is not made for joining
        ParallelMixer(a, SinkAttention(16, 4, 2, 8, 8, 0.5, None))


@pytest.mark.parametrize("dims,base,bands", [(8, 10000.0, (3.0, 1.0, 3.0, 64)), (6, 300.0, (1.5, 0.5, 2.0, 20)),
                                             (32, 1e6, (8.0, 1.0, 4.0, 4096)), (64, 20000.0, (40.0, 2.0, 2.0, 512)), (16, 50.0, None)])
def test_banded_frequencies_of_the_rotary_part_are_the_plain_ones(dims, base, bands):
    from dispec_b200.parts.rotary import RotaryEncoding
    enc = RotaryEncoding(dims, base, layout="interleaved", exact_table=True, banded=bands)
    enc.prepare("cpu")
    rot = {"dims": dims, "base": base}
    if bands:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), bands))
    if not bands or bands[1] < bands[2]:
        freq = plain.frequencies(rot)
    else:  # no band between the two: kept or divided
        f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
        freq = torch.where(2 * math.pi / f > bands[3] / bands[1], f / bands[0], f)
    got = enc.rotation()
    assert got.layout == "interleaved" and got.rotary_dim == dims and got.magnitude == 1.0
    assert (got.inv_freq.double() - freq).abs().max() <= 1e-7 * freq.abs().max()


def test_window_groups_keep_the_pages_of_the_first_tokens():
    """Over thousands of admissions, portions and releases: pages of kept first positions stay until the
    request ends, pages behind the window come back, the quota promised at admission suffices."""
    import random
    from dispec_b200.cache.manager import CacheGroupSpec, CacheManager
    rng = random.Random(4)
    for keep, window, page in ((3, 20, 16), (16, 9, 8), (17, 40, 8), (70, 64, 32), (0, 12, 4), (5, 1, 4)):
        spec = CacheGroupSpec.key_value(1, 8, window)
        spec = CacheGroupSpec(spec.tensors, window, 1, keep)
        cm = CacheManager([spec], page, 60, 4)
        kept = -(-keep // page)
        for n in range(60):
            total, chunk = rng.randint(1, 300), rng.randint(1, 24)
            if not cm.can_admit(total, total, chunk):
                continue
            cm.admit(n, total, total, chunk)
            pos, first = 0, None
            while pos < total:
                step = min(rng.randint(1, chunk), total - pos)
                cm.extend(n, pos + step)
                table = cm.block_table(n)
                lo = max(0, pos - window + 1)
                for j in range(pos + step):  # every key a token of this step may see is there
                    if j < keep or j >= lo:
                        assert table[j // page] >= 0
                pos += step
                cm.commit(n, pos)
                first = first or table[:min(kept, len(table))]
                for j, p in enumerate(table):
                    gone = j >= kept and (j + 1) * page <= max(0, pos - window + 1)
                    assert (p < 0) == gone, (j, pos)
                cm.check()
            if kept and first:
                assert cm.block_table(n)[:len(first)] == first
            cm.free(n)
            cm.check()
        assert cm.num_free_pages() == 60 and cm.largest_chunk() == (60 - 1 - kept) * page - window + 1


# ------------------------------------------------------------------ the plain implementation against itself
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_plain_token_by_token_equals_plain_whole_prompt(name):
    spec = bu.CONFIGS[name]
    weights = bu.random_weights(spec["config"], spec["seed"], spec["rank"])
    ids = ru.random_ids(45, spec["config"]["vocab"], 3)
    whole, _ = plain.forward(spec["config"], weights, ids)
    past, rows, start = None, [], 0
    for stop in (2, 17, 18, 19, 30, 32, 45):  # portions down to two tokens and single tokens
        logits, past = plain.forward(spec["config"], weights, ids[start:stop], pos=torch.arange(start, stop), past=past)
        rows.append(logits)
        start = stop
    assert (torch.cat(rows) - whole).abs().max() < 1e-9


def test_plain_mask_window_and_kept_keys():
    pos = torch.arange(12)
    seen = plain.visible(pos, pos, 4, 2)
    assert seen[11].nonzero().flatten().tolist() == [0, 1, 8, 9, 10, 11]
    assert seen[3].nonzero().flatten().tolist() == [0, 1, 2, 3] and seen[0].nonzero().flatten().tolist() == [0]
    assert seen[4].nonzero().flatten().tolist() == [0, 1, 2, 3, 4] and seen[6].nonzero().flatten().tolist() == [0, 1, 3, 4, 5, 6]
    assert torch.equal(plain.visible(pos, pos, 0, 0), torch.ones(12, 12).tril().bool())
    assert torch.equal(plain.visible(pos, pos, 12, 0), plain.visible(pos, pos, 0, 0))


def test_plain_short_conv_and_rotation_by_hand():
    u = torch.tensor([[1.0], [2.0], [4.0], [8.0]], dtype=plain.F)
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=plain.F)
    y, kept = plain.short_conv(u, w, torch.zeros(2, 1, dtype=plain.F))
    assert y.flatten().tolist() == [1.0, 12.0, 124.0, 248.0] and kept.flatten().tolist() == [4.0, 8.0]
    x = torch.zeros(1, 1, 6, dtype=plain.F)
    x[0, 0, 2], x[0, 0, 5] = 1.0, 7.0
    out = plain.turn_pairs(x, torch.tensor([3]), torch.tensor([0.5, 0.25], dtype=plain.F))  # pairs (0, 1), (2, 3)
    want = [0.0, 0.0, math.cos(0.75), math.sin(0.75), 0.0, 7.0]
    assert max(abs(a - b) for a, b in zip(out.flatten().tolist(), want)) < 1e-12


def test_plain_router_weighs_the_chosen_logits_only():
    W = {"r.router": torch.eye(4, dtype=plain.F), "r.router.b": torch.tensor([0.0, 0.0, 5.0, 0.0], dtype=plain.F)}
    ids, w = plain.route(torch.tensor([[3.0, 1.0, -1.0, 2.0]], dtype=plain.F), W, "r.", {"experts": 4, "top": 2})
    assert ids[0].tolist() == [2, 0]  # the bias counts
    e = math.exp(-1.0)
    assert abs(float(w[0, 0]) - 1 / (1 + e)) < 1e-12 and abs(float(w.sum()) - 1) < 1e-12
