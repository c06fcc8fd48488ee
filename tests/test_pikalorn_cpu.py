"""Pikalorn without a GPU: the configuration reader, the builder's tensor list against the one the
tests derive on their own, shared latents in the cache plan, states, the table of slowed frequencies, and
the plain implementation against itself (token by token and in portions through what it carries, against
whole prompts; each mechanism by hand)."""
import copy
import math

import pytest
import torch

import pikalorn_util as pu
import plain_pikalorn as plain
import replay_util as ru


def build(config):
    from dispec_b200.config.model_config import load_model_config
    from dispec_b200.weights.loader import build_model
    cfg = load_model_config(copy.deepcopy(config))
    return cfg, build_model(cfg)


@pytest.mark.parametrize("name", sorted(pu.CONFIGS))
def test_builder_asks_for_exactly_the_checkpoint_tensors(name):
    from dispec_b200.config.model_config import load_model_config
    config = pu.CONFIGS[name]["config"]
    cfg, m = build(config)
    assert load_model_config(cfg.to_dict()) == cfg
    req, want = m.tensor_requirements(), plain.tensor_shapes(config)
    assert {n: tuple(s.shape) for n, s in req.items()} == want
    assert [c.layer for c in m.schedule] == list(range(len(config["layers"])))


def test_caches_and_states_of_the_mixers():
    _, m = build(pu.CONFIGS["mix"]["config"])
    got = sorted((g.window, [(t.name, t.num_heads, t.width) for t in g.tensors], g.num_slots) for g in m.cache_groups)
    # the two layers that read layer 1's latents add no cache of their own
    assert got == [(0, [("key", 2, 16), ("value", 2, 16)], 1), (0, [("key", 6, 8), ("value", 6, 8)], 1),
                   (0, [("latent", 1, 32), ("rotated_key", 1, 16)], 1), (0, [("latent", 1, 48), ("rotated_key", 1, 8)], 1)]
    assert m.call_cache == [None, 1, 2, 1, None, 5, 1, 7]
    assert [c.write for c in m.schedule] == [True, True, True, False, True, True, False, True]
    assert m.placement[m.call_cache[3]] == m.placement[m.call_cache[1]] == m.placement[m.call_cache[6]]
    assert m.call_state == [(0, 1), None, None, None, (2, 3), None, None, None]
    assert [s.shape for s in m.state_needs] == [(4, 16, 24), (3, 2 * 2 * 16 + 4 * 24), (3, 8, 16), (1, 2 * 3 * 8 + 3 * 16)]
    assert all(s.dtype == "float32" for s in m.state_needs)
    _, odd = build(pu.CONFIGS["odd"]["config"])
    assert odd.call_state[1] == (0,)  # single taps leave no inputs behind


@pytest.mark.parametrize("change,word", [
    (lambda c: c["layers"][0].update(type="conv"), "not implemented"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "at most"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(scaling={"factor": 2.0}), "scaling"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "no latents"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=3), "no latents"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=16), "kv_rank"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=5.0), "rot"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not implemented"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_configuration_errors_name_the_key(change, word):
    from dispec_b200.config.model_config import ConfigError, load_model_config
    c = copy.deepcopy(pu.CONFIGS["mix"]["config"])
    change(c)
    with pytest.raises(ConfigError) as e:
        load_model_config(c)
    assert word in str(e.value)


def test_part_constructors_refuse_what_cannot_run():
    from dispec_b200.parts.attention import ConvAttention, SinkAttention
    from dispec_b200.parts.block import ParallelPreNormBlock
    from dispec_b200.parts.linear_attention import GatedDelta, Retention
    from dispec_b200.parts.parallel import ParallelMixer
    from dispec_b200.parts.state_space import StateSpaceDual
    with pytest.raises(ValueError):
        GatedDelta(16, 4, 3, 8, 8, 2, 1e-6)
    with pytest.raises(ValueError):
        GatedDelta(16, 2, 1, 513, 8, 2, 1e-6)
    with pytest.raises(ValueError):
        SinkAttention(16, 4, 2, 8, 6, 0.5, None, values="keys")
    with pytest.raises(ValueError):
        SinkAttention(16, 4, 2, 8, 8, 0.5, None, values="keys", value_mix=("source", 0))
    delta = GatedDelta(16, 4, 2, 8, 8, 2, 1e-6)
    with pytest.raises(ValueError):  # not made for joining
        ParallelPreNormBlock(16, None, Retention(16, 2, 8, 8, [0.5, 0.6], 1e-6, None))
    with pytest.raises(ValueError):  # a feed-forward without rows of its own
        ParallelPreNormBlock(16, None, delta, object())
    with pytest.raises(ValueError):  # takes no factor
        ParallelMixer(ConvAttention(16, 4, 2, 8, 8, 0.5, None), delta, 1.0, 0.5)
    with pytest.raises(ValueError):
        ParallelMixer(SinkAttention(16, 4, 2, 8, 8, 0.5, None), StateSpaceDual(16, 4, 8, 8, 2, 2, 1, 1e-6), 2.0, 1.0)


@pytest.mark.parametrize("dims,base,slowed", [(16, 10000.0, (4.0, 64, 32.0, 1.0)), (6, 300.0, (1.5, 20, 4.0, 0.5)),
                                              (64, 1e6, (40.0, 4096, 32.0, 1.0)), (8, 50.0, None), (4, 9.0, (3.0, 2, 1.0, 1.0))])
def test_slowed_frequencies_of_the_rotary_part_are_the_plain_ones(dims, base, slowed):
    from dispec_b200.parts.rotary import RotaryEncoding
    enc = RotaryEncoding(dims, base, layout="interleaved", exact_table=True, slowed=slowed)
    enc.prepare("cpu")
    rot = {"dims": dims, "base": base}
    if slowed:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), slowed))
    freq, mag = plain.frequencies(rot)
    got = enc.rotation()
    assert got.layout == "interleaved" and got.rotary_dim == dims and abs(got.magnitude - mag) < 1e-12
    assert (got.inv_freq.double() - freq).abs().max() <= 1e-7 * freq.abs().max()


# ------------------------------------------------------------------ the plain implementation against itself
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_plain_token_by_token_equals_plain_whole_prompt(name):
    spec = pu.CONFIGS[name]
    weights = pu.random_weights(spec["config"], spec["seed"])
    ids = ru.random_ids(45, spec["config"]["vocab"], 3)
    whole, _ = plain.forward(spec["config"], weights, ids)
    past, rows, start = None, [], 0
    for stop in (2, 17, 18, 19, 30, 32, 45):  # portions down to two tokens and single tokens
        logits, past = plain.forward(spec["config"], weights, ids[start:stop], pos=torch.arange(start, stop), past=past)
        rows.append(logits)
        start = stop
    assert (torch.cat(rows) - whole).abs().max() < 1e-9


def test_plain_sink_takes_its_share_and_gives_nothing():
    q = torch.tensor([[[2.0]], [[2.0]]], dtype=plain.F)
    k, v = torch.tensor([[[1.0]], [[0.5]]], dtype=plain.F), torch.tensor([[[10.0]], [[-4.0]]], dtype=plain.F)
    pos = torch.arange(2)
    o = plain.sink_softmax_attention(q, k, v, pos, pos, 0.5, torch.tensor([0.3], dtype=plain.F))
    e = [math.exp(1.0), math.exp(0.5), math.exp(0.3)]
    assert abs(float(o[0]) - 10 * e[0] / (e[0] + e[2])) < 1e-12
    assert abs(float(o[1]) - (10 * e[0] - 4 * e[1]) / sum(e)) < 1e-12


def test_plain_rotation_layouts_and_magnitude_by_hand():
    x = torch.arange(1.0, 7.0, dtype=plain.F).view(1, 1, 6)
    rot = {"dims": 4, "base": 16.0}  # frequencies 1 and 1/4
    pos = torch.tensor([2])
    c, s = [math.cos(2.0), math.cos(0.5)], [math.sin(2.0), math.sin(0.5)]
    inter = plain.turn(x, pos, rot, True).flatten().tolist()
    want = [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 5.0, 6.0]
    assert max(abs(a - b) for a, b in zip(inter, want)) < 1e-12
    half = plain.turn(x, pos, rot, False).flatten().tolist()
    want = [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 5.0, 6.0]
    assert max(abs(a - b) for a, b in zip(half, want)) < 1e-12
    # bands in front of the first pair: it stays, every other is divided by the factor; lengths times the magnitude
    slow = dict(rot, scaling={"factor": 2.0, "original": 1e-3, "fast": 32.0, "slow": 1.0})
    f, mag = plain.frequencies(slow)
    assert f.tolist() == [1.0, 0.125]
    assert abs(mag - (0.1 * math.log(2.0) + 1)) < 1e-15
    y = plain.turn(x, pos, slow, True)
    assert abs(float(y[..., :4].norm() / x[..., :4].norm()) - mag) < 1e-12 and y[0, 0, 4:].tolist() == [5.0, 6.0]


def test_plain_delta_rule_replaces_what_a_key_held():
    """beta 1 and no decay: writing a second value under the same key leaves only the second one; a read with an
    orthogonal query sees nothing; decay and read-out see the current write."""
    one = torch.ones(3, 1, dtype=plain.F)
    k = torch.tensor([[1.0, 0.0], [1.0, 0.0], [0.0, 1.0]], dtype=plain.F).view(3, 1, 2)
    v = torch.tensor([[5.0], [7.0], [9.0]], dtype=plain.F).view(3, 1, 1)
    o, S = plain.delta_scan(k, k, v, one, one, torch.zeros(1, 2, 1, dtype=plain.F))
    assert o.flatten().tolist() == [5.0, 7.0, 9.0] and S.flatten().tolist() == [7.0, 9.0]
    o, S = plain.delta_scan(k.flip(-1), k, v, one, one, torch.zeros(1, 2, 1, dtype=plain.F))
    assert o.flatten().tolist() == [0.0, 0.0, 7.0]
    half = 0.5 * one
    o, S = plain.delta_scan(k, k, v, half, half, torch.zeros(1, 2, 1, dtype=plain.F))
    # 2.5; then S = 1.25, u = (7 - 1.25) / 2
    assert o.flatten().tolist() == [2.5, 1.25 + 2.875, 4.5]


def test_plain_short_conv_by_hand():
    u = torch.tensor([[1.0], [2.0], [4.0], [8.0]], dtype=plain.F)
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=plain.F)
    y, kept = plain.short_conv(u, w, torch.zeros(2, 1, dtype=plain.F))
    assert y.flatten().tolist() == [1.0, 12.0, 124.0, 248.0] and kept.flatten().tolist() == [4.0, 8.0]


def test_plain_values_are_the_projected_keys():
    """One key: whatever the rotation and the norm, the result is its raw projection times the share the sink leaves."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "rot": {"dims": 2, "base": 10.0}}
    e = torch.eye(2, dtype=plain.F)
    W = {"q": e, "k": 3 * e, "q.b": torch.zeros(2), "k.b": torch.tensor([0.5, -1.0]), "q.norm": torch.ones(2), "k.norm": 2 * torch.ones(2),
         "sink": torch.tensor([-1e9]), "g": torch.zeros(2, 2), "o": e, "o.b": torch.tensor([100.0, 0.0])}
    W = {k: v.to(plain.F) for k, v in W.items()}
    y, _ = plain.attention(torch.tensor([[1.0, 2.0]], dtype=plain.F), W, "", m, 1e-6, torch.tensor([5]), None)
    assert (y - torch.tensor([[100.0 + 0.5 * 3.5, 0.5 * 5.0]], dtype=plain.F)).abs().max() < 1e-9
