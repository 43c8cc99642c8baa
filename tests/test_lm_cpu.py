"""Layered models without a device: the restatement's mechanisms against hand-worked cases, the registry and
the file readers' refusals, the block bookkeeping of the paged cache."""
import json
import subprocess
from pathlib import Path

import numpy as np
import pytest

import latent_oracle as la
import lenedra_oracle as le
import lm_oracle as lo
import lm_util
import zevilorn_oracle as ze

ROOT = Path(__file__).resolve().parents[1]


# ---- the restatement ----------------------------------------------------------------------------------
def test_sinusoid_entries():
    s = lo.sinusoid([0, 3], 6)
    assert np.allclose(s[0], [0, 1, 0, 1, 0, 1])
    f = [1.0, 10000 ** (-2 / 6), 10000 ** (-4 / 6)]
    assert np.allclose(s[1], [np.sin(3 * f[0]), np.cos(3 * f[0]), np.sin(3 * f[1]), np.cos(3 * f[1]), np.sin(3 * f[2]), np.cos(3 * f[2])])


def test_window_edge_and_bias():
    assert lo.window_mask([5], range(8), 3)[0].tolist() == [False] * 3 + [True] * 3 + [False] * 2
    assert lo.window_mask([0, 1], [0, 1], 1).tolist() == [[True, False], [False, True]]
    assert np.allclose(lo.alibi_slopes(4), [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8])
    assert np.allclose(lo.distance_bias(np.zeros((1, 3)), [2], [0, 1, 2], 0.5), [[-1.0, -0.5, 0.0]])


def test_sink_takes_its_share():
    p = lo.softmax_with_sink(np.array([[0.0, 0.0, 5.0]]), np.array([[True, True, False]]))
    assert np.allclose(p, [[1 / 3, 1 / 3, 0]])
    p = lo.softmax_with_sink(np.array([[-800.0, 800.0]]), np.array([[True, True]]))
    assert np.allclose(p, [[0, 1]])


def test_query_temperature_steps():
    t = lo.query_temperature([0, 8, 9, 18, 19], 0.5, 10)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 2, 2, 3]))


def test_norm_and_activation():
    x = np.array([[3.0, -4.0]])
    assert np.allclose(lo.rms_norm(x, np.array([1.0, 2.0]), 0.5), x / np.sqrt(13.0) * [1, 2])
    assert np.allclose(lo.gelu_tanh(np.array([0.0, 1.0, -1.0])), [0.0, 0.841192, -0.158808], atol=1e-6)


@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "plain", "latent", "latent_odd", "latent_wide", "latent_full", "streams", "streams_odd", "streams_wide",
                                  "streams_full", "loops", "loops_odd", "loops_wide", "loops_full", "loops_windows"])
def test_portions_change_nothing(synth, tmp_path, name):
    cfg, w, _ = lm_util.build(synth, tmp_path, name)
    m = lm_util.model(cfg, w)
    tokens = np.random.default_rng(3).integers(0, cfg["vocab"], 60)
    whole = m.forward(tokens)
    state = m.new_state()
    parts = [m.forward(tokens[a:b], state) for a, b in lm_util.cut(60, [2, 17, 1, 5])]
    assert np.allclose(np.concatenate(parts), whole, atol=1e-9)


def test_shared_weights_keep_their_own_cache(synth, tmp_path):
    cfg, w, _ = lm_util.build(synth, tmp_path, "mixed")
    m = lo.Model(cfg, w)
    st = m.new_state()
    m.forward([1, 2, 3], st)
    assert not np.allclose(st["caches"][0]["k"], st["caches"][2]["k"]) and not any(n.startswith("l2.") for n in w)


def test_every_setting_shows_in_the_logits(synth, tmp_path):
    """Configurations of the end-to-end tests are such that a setting read wrongly moves the logits."""
    cfg, w, _ = lm_util.build(synth, tmp_path, "latent")
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 90)
    want = lm_util.reference(cfg, w, t)

    def moved(change, w2=None):
        other = json.loads(json.dumps(cfg))
        change(other["layers"])
        assert lm_util.error(lm_util.reference(other, w2 or w, t), want) > 100 * lm_util.TOL[0]
    moved(lambda l: l[1]["mixer"]["mask"].update(size=18))
    moved(lambda l: l[3]["mixer"]["mask"].update(size=71))
    moved(lambda l: l[0]["mixer"]["rot"].update(base=10100.0))
    moved(lambda l: l[0]["mixer"].update(scale=0.18))
    for k, v in (("factor", 3.0), ("original", 32), ("fast", 4.0), ("slow", 3.0)):
        moved(lambda l: l[1]["mixer"]["rot"]["scaling"].update({k: v}))
    moved(lambda l: l[1]["mixer"]["rot"].pop("scaling"))
    moved(lambda l: l[1]["mlp"]["router"].update(top=1))
    moved(lambda l: l[4]["mlp"]["expert"].update(limit=0.5))
    moved(lambda l: l[1].update(type="latent_attention"))                # no gate
    for name in ("l0.mlp.act", "l2.mix.uk", "l2.mix.uv", "l3.mix.g", "l0.mix.dkv.norm", "l4.mlp.e3.up", "final.norm"):
        w2 = dict(w)
        w2[name] = w[name][::-1]
        moved(lambda l: None, w2)


# ---- the latents' restatement -----------------------------------------------------------------------------
def test_rotation_by_hand():
    rot = {"dims": 4, "base": 100.0}
    f, mul = la.frequencies(rot)
    assert np.allclose(f, [1.0, 0.1]) and mul == 1.0
    x = np.array([[1.0, 2.0, 3.0, 4.0]] * 2)
    y = la.rotate(x, [0, 5], rot)
    assert np.allclose(y[0], x[0])
    c, s = np.cos([5.0, 0.5]), np.sin([5.0, 0.5])
    assert np.allclose(y[1], [1 * c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + 1 * s[0], 4 * c[1] + 2 * s[1]])


def test_frequency_scaling_by_hand():
    # dims 8, base 10^4: f = 1, .1, .01, .001. Turns within 200 positions: 31.8, 3.18, 0.318, 0.0318
    f, mul = la.frequencies({"dims": 8, "base": 10000.0, "scaling": {"factor": 5.0, "original": 200, "fast": 10.0, "slow": 0.1}})
    at = lambda t: 8 * np.log(200 / (2 * np.pi * t)) / (2 * np.log(10000.0))
    lo, hi = np.floor(at(10.0)), np.ceil(at(0.1))
    assert (lo, hi) == (0, 3)
    ramp = np.arange(4) / 3
    plain = np.array([1, 0.1, 0.01, 0.001])
    assert np.allclose(f, plain * (1 - ramp) + plain / 5 * ramp) and np.isclose(mul, 1 + 0.1 * np.log(5.0))
    f, _ = la.frequencies({"dims": 8, "base": 10000.0, "scaling": {"factor": 5.0, "original": 2, "fast": 10.0, "slow": 9.0}})
    assert np.allclose(f, plain / 5 * np.array([0, 1, 1, 1]) + plain * np.array([1, 0, 0, 0]))     # both ends below the first pair: a step


def test_visibility_and_softmax():
    assert la.visible([5], range(8), 3)[0].tolist() == [False] * 3 + [True] * 3 + [False] * 2
    assert la.visible([5], range(8), None)[0].tolist() == [True] * 6 + [False] * 2
    assert np.allclose(la.softmax(np.array([[0.0, np.log(3.0), 9.0]]), np.array([[True, True, False]])), [[0.25, 0.75, 0.0]])


def test_poly_norm_by_hand():
    z = np.array([[1.0, -2.0]])
    n = lambda v: v / np.sqrt((v ** 2).mean() + 0.5)
    assert np.allclose(la.poly_norm(z, [2.0, 3.0, 5.0, 7.0], 0.5), 2 * n(z) + 3 * n(z ** 2) + 5 * n(z ** 3) + 7)


def test_routing_and_experts_by_hand():
    ids, wt = la.route(np.array([[1.0, 0.0]]), np.array([[0.0, 9.0], [2.0, 0.0], [2.0, 0.0], [1.0, 0.0]]), 2)
    e = np.exp([0.0, 2.0, 2.0, 1.0])
    assert ids.tolist() == [[1, 2]] and np.allclose(wt, e[1] / e.sum())                  # not renormalised; a tie goes to the lower index
    g, u = np.array([5.0, -5.0, 1.0]), np.array([3.0, -3.0, 0.5])
    sg = lambda z: 1 / (1 + np.exp(-1.702 * z))
    assert np.allclose(la.clamped_glu(g, u, 2.0), [2 * sg(2.0) * 3, -5 * sg(-5.0) * -1, sg(1.0) * 1.5])
    w = {"router": np.array([[1.0], [2.0]]), **{f"e{i}.{n}": np.array([[float(i + 1)]]) for i in range(2) for n in ("gate", "up", "down")}}
    out = la.experts(np.array([[1.0]]), w, {"router": {"experts": 2, "top": 1}, "expert": {"limit": 9.0}})
    assert np.allclose(out, np.exp(2) / (np.exp(1) + np.exp(2)) * 2 * (2 * sg(2.0) * 3))


def test_a_layer_reads_the_named_cache(synth, tmp_path):
    cfg, w, _ = lm_util.build(synth, tmp_path, "latent")
    m = lm_util.model(cfg, w)
    st = m.new_state()
    m.forward([1, 2, 3], st)
    assert st["caches"][2] == {} and len(st["caches"][0]["c"]) == 3 and "l2.mix.dkv" not in w


# ---- the restatement of streams, kept windows, chunks, the delta rule and grouped routing ----------------
def test_kept_window_and_chunks_by_hand():
    seen = le.window_with_kept([6], range(9), 2, 3)[0]
    assert seen.tolist() == [True] * 3 + [False] * 2 + [True] * 2 + [False] * 2
    assert le.window_with_kept([1], range(4), 1, 3)[0].tolist() == [True, True, False, False]          # kept, but not before its time
    assert le.same_chunk([3, 4, 7], range(8), 4).tolist() == [[True] * 4 + [False] * 4, [False] * 4 + [True] + [False] * 3, [False] * 4 + [True] * 4]


def test_learned_sink_by_hand():
    p = le.weights_over(np.array([[0.0, np.log(2.0), 9.0]]), np.array([[True, True, False]]), np.log(5.0))
    assert np.allclose(p, [[1 / 8, 2 / 8, 0]])
    assert np.allclose(le.weights_over(np.array([[-900.0]]), np.array([[True]]), -900.0), [[0.5]])


def test_delta_rule_by_hand():
    S = np.array([[2.0], [4.0]])
    o = le.delta_rule(np.array([[1.0, 2.0]]), np.array([[0.6, 0.8]]), np.array([[5.0]]), np.array([[0.5, 0.25]]), np.array([0.5]), S)
    u = 0.5 * (5 - (0.6 * 1 + 0.8 * 1))                                       # the decayed state is (1, 1)
    assert np.allclose(S, [[1 + 0.6 * u], [1 + 0.8 * u]]) and np.allclose(o, [[S[0, 0] + 2 * S[1, 0]]])       # the read sees the write


def test_causal_convolution_by_hand():
    x, taps = np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 1.0]])
    y, past = le.causal_conv(x, taps, np.zeros((1, 1)))
    assert np.allclose(y, le.silu(np.array([[1.0], [12.0], [23.0]]))) and past.tolist() == [[3.0]]
    y, past = le.causal_conv(x, taps[:, 1:], np.zeros((0, 1)))
    assert np.allclose(y, le.silu(x)) and past.shape == (0, 1)


def test_grouped_choice_by_hand():
    z = np.log(np.array([[0.4, 0.1, 0.2, 0.3]]))
    w = {"router": np.eye(4), "correction": np.array([-1.0, -1.0, -2.0, -1.05])}
    r = {"groups": {"count": 2, "keep": 1}, "top": 2, "scale": 3.0}
    ids, p = le.route(z, w, r)                                                # choice: -0.6 -0.9 | -1.8 -0.75
    assert ids.tolist() == [[0, 1]] and np.allclose(p, [[3 * 0.8, 3 * 0.2]])
    ids, _ = le.route(z, w, {**r, "groups": {"count": 2, "keep": 2}})
    assert ids.tolist() == [[0, 3]]


def test_streams_by_hand():
    x = np.array([[[1.0]], [[10.0]]])
    assert le.read_streams(x, np.array([2.0, 3.0])).tolist() == [[32.0]]
    y = le.write_streams(x, np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([5.0, 6.0]), np.array([[100.0]]))
    assert y.tolist() == [[[1 + 30 + 500]], [[2 + 40 + 600]]]                  # mix is [from, to]


def test_every_setting_of_a_design_with_streams_shows(synth, tmp_path):
    cfg, w, _ = lm_util.build(synth, tmp_path, "streams")
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 90)
    want = lm_util.reference(cfg, w, t)

    def moved(change, w2=None):
        other = json.loads(json.dumps(cfg))
        change(other, other["layers"])
        assert lm_util.error(lm_util.reference(other, w2 or w, t), want) > 100 * lm_util.TOL[0]
    moved(lambda c, l: l[0]["mixer"]["mask"].update(size=18))
    moved(lambda c, l: l[0]["mixer"]["mask"].update(keep_first=4))
    moved(lambda c, l: l[0]["mixer"].update(scale=0.3))
    moved(lambda c, l: l[1]["mixer"]["left"]["mask"].update(size=38))
    moved(lambda c, l: l[1]["mixer"]["left"].update(scale=0.3))
    moved(lambda c, l: l[1]["mixer"].update(left_scale=0.9))
    moved(lambda c, l: l[3]["mixer"].update(right_scale=1.1))
    moved(lambda c, l: l[1]["mlp"]["router"].update(top=2))
    moved(lambda c, l: l[1]["mlp"]["router"].update(scale=1.2))
    moved(lambda c, l: l[1]["mlp"]["router"]["groups"].update(keep=1))
    moved(lambda c, l: l[1]["mlp"]["router"].update(experts=6, identity=4))    # the last expert becomes an identity
    moved(lambda c, l: c["embedding"].update(scale=2.5))
    moved(lambda c, l: c.update(logit_softcap=5.0))
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.o.b", "l0.mix.q.norm", "l0.mix.k.norm", "l1.mix.left.sink", "l1.mix.left.v.b", "l1.mix.right.q.conv", "l1.mix.right.v.conv",
                 "l1.mix.right.A_log", "l1.mix.right.dt_bias", "l1.mix.right.b", "l1.mix.right.norm", "l3.mix.right.a2", "l3.mix.right.g1", "l1.mlp.correction", "l1.mlp.shared.up",
                 "l1.hc1.in", "l1.hc2.out", "l3.norm1", "final.norm"):
        w2 = dict(w)
        w2[name] = np.roll(w[name][::-1], 1, 0) if len(w[name]) == 3 else w[name][::-1]
        moved(lambda c, l: None, w2)
    w2 = dict(w)
    w2["l1.hc1.mix"] = w["l1.hc1.mix"].T
    moved(lambda c, l: None, w2)


# ---- the restatement of looped layers, gates, talking heads, the minimal recurrence and sigmoid routing ------
def test_rotation_of_neighbours_and_halves_by_hand():
    f = ze.frequencies({"dims": 4, "base": 100.0})
    assert np.allclose(f, [1.0, 0.1])
    x = np.array([[[1.0, 2.0, 3.0, 4.0, 9.0]]] * 2)
    c, s = np.cos([5.0, 0.5]), np.sin([5.0, 0.5])
    y = ze.rotate_neighbours(x, [0, 5], f)
    assert np.allclose(y[0], x[0]) and np.allclose(y[1, 0], [c[0] - 2 * s[0], 2 * c[0] + s[0], 3 * c[1] - 4 * s[1], 4 * c[1] + 3 * s[1], 9])
    y = ze.rotate_halves(x, [0, 5], f)
    assert np.allclose(y[1, 0], [c[0] - 3 * s[0], 2 * c[1] - 4 * s[1], 3 * c[0] + s[0], 4 * c[1] + 2 * s[1], 9])


def test_frequency_scalings_by_hand():
    tau = 2 * np.pi
    # turns within 100 positions: 8 (stays), 2 (a third of the way from 1 to 4), 0.5 (stretched)
    f = np.array([8, 2, 0.5]) * tau / 100
    s = {"factor": 5.0, "low": 1.0, "high": 4.0, "original": 100}
    assert np.allclose(ze.scale_banded(f, s), f * [1, (2 / 3) / 5 + 1 / 3, 1 / 5])
    assert np.allclose(ze.scale_linear(f, {"factor": 4.0}), f / 4)


def test_cap_and_mixed_heads_by_hand():
    assert np.allclose(ze.soft_cap(np.array([1.0, -50.0]), 2.0), [2 * np.tanh(0.5), -2])
    s = np.array([[[1.0, 2.0]], [[10.0, 20.0]]])                              # [head, query, key]
    assert np.allclose(ze.mix_heads(s, np.array([[1.0, 3.0], [0.0, -1.0]])), [[[31, 62]], [[-10, -20]]])
    p = ze.weights_over(np.log(np.array([[[1.0, 3.0, 9.0]]])), ze.window([5], [4, 5, 6], 2), [0.0])
    assert np.allclose(p, [[[1 / 5, 3 / 5, 0]]])
    assert ze.window([5], range(8), 3)[0].tolist() == [False] * 3 + [True] * 3 + [False] * 2


def test_convolution_without_activation_by_hand():
    y, past = ze.causal_conv(np.array([[1.0], [2.0], [3.0]]), np.array([[100.0, 10.0, 1.0]]), np.zeros((2, 1)))
    assert y.ravel().tolist() == [1, 12, 123] and past.ravel().tolist() == [2, 3]


def test_minimal_recurrence_by_hand():
    assert np.allclose(ze.candidate(np.array([0.0, 2.0, -1.0])), [0.5, 2.5, ze.sigmoid(-1.0)])
    S = ze.gated_scan(np.array([[0.25], [1.0], [0.5]]), np.array([[4.0], [3.0], [1.0]]), np.array([8.0]))
    assert S.ravel().tolist() == [7.0, 3.0, 2.0]


def test_groups_by_their_two_best_by_hand():
    z = np.log(np.array([[0.9, 0.1, 0.1, 0.5, 0.55, 0.1]]) / (1 - np.array([[0.9, 0.1, 0.1, 0.5, 0.55, 0.1]])))
    r = {"groups": {"count": 2, "keep": 1}, "top": 2}
    ids, p = ze.route(z, {"router": np.eye(6)}, r)                             # 0.9 + 0.1 against 0.55 + 0.5
    assert ids.tolist() == [[4, 3]] and np.allclose(p, [[0.55, 0.5]])
    ids, p = ze.route(z, {"router": np.eye(6)}, {"top": 2})
    assert ids.tolist() == [[0, 4]] and np.allclose(p, [[0.9, 0.55]])
    assert np.allclose(ze.gelu_erf(np.array([0.0, 1.0, -1.0])), [0, 0.8413447, -0.1586553])


def test_loop_order_by_hand():
    cfg = {"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 3}}
    assert ze.runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert ze.runs({"layers": [0] * 2}) == [(0, False), (1, False)]


def test_every_setting_of_a_design_with_loops_shows(synth, tmp_path):
    cfg, w, _ = lm_util.build(synth, tmp_path, "loops")
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 110)
    want = lm_util.reference(cfg, w, t)

    def moved(change, w2=None):
        other = json.loads(json.dumps(cfg))
        change(other, other["layers"])
        assert lm_util.error(lm_util.reference(other, w2 or w, t), want) > 100 * lm_util.TOL[0]
    mixer = lambda l, i: l[i]["mixer"]
    moved(lambda c, l: mixer(l, 0)["mask"].update(size=36))
    moved(lambda c, l: mixer(l, 3)["mask"].update(size=71))
    moved(lambda c, l: mixer(l, 2)["left"]["mask"].update(size=22))
    moved(lambda c, l: mixer(l, 0).update(softcap=5.0))
    for k in (0, 1):
        moved(lambda c, l: mixer(l, k).update(scale=0.3))
    moved(lambda c, l: mixer(l, 2)["left"].update(scale=0.3))
    moved(lambda c, l: mixer(l, 0)["rot"].update(base=450.0))
    moved(lambda c, l: mixer(l, 0)["rot"].update(dims=18))
    moved(lambda c, l: mixer(l, 1)["rot"].update(base=9000.0))
    moved(lambda c, l: mixer(l, 2)["left"]["rot"].update(dims=10))
    for k, v in (("factor", 2.0), ("low", 0.5), ("high", 8.0), ("original", 50)):
        moved(lambda c, l: mixer(l, 0)["rot"]["scaling"].update({k: v}))
    moved(lambda c, l: mixer(l, 2)["left"]["rot"]["scaling"].update(factor=2.0))
    moved(lambda c, l: mixer(l, 2)["left"]["rot"].pop("scaling"))
    moved(lambda c, l: l[0]["mlp"]["router"].update(top=1))
    moved(lambda c, l: l[0]["mlp"]["router"]["groups"].update(keep=4))
    moved(lambda c, l: l[3]["mlp"]["router"].pop("groups"))
    for loop in ((1, 4, 2), (0, 4, 3), (1, 3, 3), (2, 4, 3)):
        moved(lambda c, l: c.update(loop=dict(zip(("start", "stop", "times"), loop))))
    for name in ("l0.mix.q.b", "l0.mix.v.b", "l0.mix.o.b", "l0.mix.k.conv", "l0.mix.v.conv", "l0.mix.talk", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.uv",
                 "l1.mix.sink", "l1.mix.g", "l2.mix.left.g", "l2.mix.left.out", "l2.mix.right.z", "l2.mix.right.z.b", "l2.mix.right.x.b", "l2.mix.right.g", "l2.mix.right.out",
                 "l0.rg1", "l0.rg2.b", "l1.mlp.e2.up", "l3.norm1", "final.norm"):
        w2 = dict(w)
        w2[name] = w[name][::-1]
        moved(lambda c, l: None, w2)
    w2 = dict(w)
    w2["l0.mix.talk"] = w["l0.mix.talk"].T
    moved(lambda c, l: None, w2)


# ---- registry and readers ------------------------------------------------------------------------------
def test_registry_knows_its_classes(pkg):
    assert pkg.lib.cml_lm_known(b"Situlorn") == 1 and pkg.lib.cml_lm_known(b"Lenedra") == 1 and pkg.lib.cml_lm_known(b"Zevilorn") == 1
    assert pkg.lib.cml_lm_known(b"Rarolorn") == 1 and pkg.lib.cml_lm_known(b"llama") == 1
    assert pkg.lib.cml_lm_known(b"nothing") == 0 and pkg.lib.cml_lm_known(None) == 0
    o = pkg.lib.cml_lm_default_options()
    assert (o.dtype, o.max_tokens, o.max_sequences, o.max_step_rows) == (pkg.DTYPE_BFLOAT16, 8192, 8, 0)


def _load(pkg, folder, **kw):
    o = pkg.LMOptions(kw.get("dtype", pkg.DTYPE_BFLOAT16), kw.get("max_tokens", 64), kw.get("max_sequences", 1), 0)
    return pkg.lib.cml_lm_load(str(folder).encode(), o)


def test_load_refusals(pkg, synth, tmp_path):
    """Everything here is refused while reading config.json, before a device is needed."""
    cfg, w, folder = lm_util.build(synth, tmp_path, "plain")

    def with_config(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        (folder / "config.json").write_text(json.dumps(c))
        assert not _load(pkg, folder)

    with_config(lambda c: c.pop("architecture"))
    with_config(lambda c: c.update(architecture="Other"))
    with_config(lambda c: c.pop("width"))
    with_config(lambda c: c.pop("norm"))
    with_config(lambda c: c.update(layers=[]))
    with_config(lambda c: c["layers"][0].update(type="recurrent"))
    with_config(lambda c: c["layers"][0]["mixer"].pop("scale"))
    with_config(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    with_config(lambda c: c["layers"][0]["mixer"]["mask"].update(size=0))
    with_config(lambda c: c["layers"][0]["mixer"]["q_temp"].pop("every"))
    with_config(lambda c: c["layers"][0]["mlp"].update(kind="sparse"))
    with_config(lambda c: c["layers"][1].update(weights_of=0))          # another shape
    with_config(lambda c: c["layers"][1].update(weights_of=7))
    for text in ("", "{", '{"architecture": "Rarolorn",}', '{"architecture": "Rarolorn"} x', "[" * 100, '{"a": "\\ud800"}', '{"a": 1e999}'):
        (folder / "config.json").write_text(text)
        assert not _load(pkg, folder)
    (folder / "config.json").unlink()
    assert not _load(pkg, folder) and not _load(pkg, tmp_path / "absent")
    (folder / "config.json").write_text(json.dumps(cfg))
    assert not _load(pkg, folder, dtype=pkg.DTYPE_BFLOAT16 + 1) and not _load(pkg, folder, max_tokens=0) and not _load(pkg, folder, max_sequences=0)


def test_latent_load_refusals(pkg, synth, tmp_path):
    cfg, w, folder = lm_util.build(synth, tmp_path, "latent")
    mixer = lambda c, i: c["layers"][i]["mixer"]

    def with_config(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        (folder / "config.json").write_text(json.dumps(c))
        assert not _load(pkg, folder)

    for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale", "rot"):
        with_config(lambda c: mixer(c, 0).pop(key))
    with_config(lambda c: c["layers"][0].update(type="attention"))                        # another design's mixer
    with_config(lambda c: c["layers"][0].update(type="latent_attention_3"))
    with_config(lambda c: mixer(c, 0)["rot"].update(dims=6))                                 # not rot_dim
    with_config(lambda c: (mixer(c, 0)["rot"].update(dims=7), mixer(c, 0).update(rot_dim=7)))
    with_config(lambda c: mixer(c, 0)["rot"].update(base=1.0))
    with_config(lambda c: mixer(c, 1)["rot"]["scaling"].pop("slow"))
    with_config(lambda c: mixer(c, 1)["rot"]["scaling"].update(factor=0))
    with_config(lambda c: mixer(c, 1)["mask"].update(size=0))
    with_config(lambda c: mixer(c, 0).update(kv_rank=513))
    for j in (-1, 2, 3, 4, 9, 1, 0.5):                                                       # itself or later, unlike latents, not a layer
        with_config(lambda c: mixer(c, 2).update(kv_from=j))
    with_config(lambda c: mixer(c, 4).update(kv_from=2))                                     # has no latents of its own
    with_config(lambda c: mixer(c, 2)["rot"].update(base=500.0))
    with_config(lambda c: c["layers"][1]["mlp"]["router"].update(top=6))
    with_config(lambda c: c["layers"][1]["mlp"]["router"].update(experts=0))
    with_config(lambda c: c["layers"][1]["mlp"].pop("expert"))
    with_config(lambda c: c["layers"][1]["mlp"].update(kind="dense"))
    with_config(lambda c: c["layers"][0]["mlp"].update(ff=-1))


def test_streams_load_refusals(pkg, synth, tmp_path):
    cfg, w, folder = lm_util.build(synth, tmp_path, "streams")
    mixer = lambda c, i: c["layers"][i]["mixer"]

    def with_config(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        (folder / "config.json").write_text(json.dumps(c))
        assert not _load(pkg, folder)

    with_config(lambda c: c.pop("streams"))
    with_config(lambda c: c.update(streams=0))
    with_config(lambda c: c.update(streams=9))
    with_config(lambda c: c["layers"][0].update(type="latent_attention"))
    with_config(lambda c: mixer(c, 0)["mask"].update(keep_first=-1))
    with_config(lambda c: mixer(c, 0).update(vdim=25))                           # values are keys
    for side in ("left", "right"):
        for key in ("heads", "kv_heads", "dim", "vdim"):
            with_config(lambda c: mixer(c, 1)[side].pop(key))
        with_config(lambda c: mixer(c, 1).pop(side))
        with_config(lambda c: mixer(c, 1).pop(side + "_scale"))
    with_config(lambda c: mixer(c, 1)["left"]["mask"].update(size=0))
    with_config(lambda c: mixer(c, 1)["right"].update(conv=0))
    with_config(lambda c: mixer(c, 1)["right"].update(kv_heads=3))
    with_config(lambda c: mixer(c, 1)["right"].update(dim=257))
    router = lambda c: c["layers"][1]["mlp"]["router"]
    with_config(lambda c: router(c).update(identity=-1))
    with_config(lambda c: router(c).update(top=11))
    with_config(lambda c: router(c)["groups"].update(count=3))                   # does not divide the outputs
    with_config(lambda c: router(c)["groups"].update(keep=6))
    with_config(lambda c: router(c).update(top=5))                               # more than the kept groups hold
    with_config(lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0))


def test_loops_load_refusals(pkg, synth, tmp_path):
    cfg, w, folder = lm_util.build(synth, tmp_path, "loops")
    mixer = lambda c, i: c["layers"][i]["mixer"]

    def with_config(change):
        c = json.loads(json.dumps(cfg))
        change(c)
        (folder / "config.json").write_text(json.dumps(c))
        assert not _load(pkg, folder)

    for loop in ({"start": 1, "stop": 6, "times": 2}, {"start": -1, "stop": 2, "times": 2}, {"start": 3, "stop": 2, "times": 2}, {"start": 0, "stop": 2, "times": 0}, {"start": 0, "stop": 2},
                 {"start": 0, "stop": 5, "times": 100000}):
        with_config(lambda c: c.update(loop=loop))
    for key in ("heads", "kv_heads", "dim", "vdim", "scale", "conv", "rot"):
        with_config(lambda c: mixer(c, 0).pop(key))
    with_config(lambda c: mixer(c, 0).update(conv=0))
    with_config(lambda c: mixer(c, 0).update(conv=65))
    with_config(lambda c: mixer(c, 0).update(softcap=-1.0))
    with_config(lambda c: mixer(c, 0).update(heads=999, kv_heads=1))              # more than can mix their scores
    with_config(lambda c: mixer(c, 0)["mask"].update(size=0))
    for dims in (0, 7, 26, -2):
        with_config(lambda c: mixer(c, 0)["rot"].update(dims=dims))
    for key in ("factor", "low", "high", "original"):
        with_config(lambda c: mixer(c, 0)["rot"]["scaling"].pop(key))
    with_config(lambda c: mixer(c, 0)["rot"]["scaling"].update(high=1.0))
    with_config(lambda c: mixer(c, 2)["left"]["rot"]["scaling"].update(factor=0))
    for key in ("q_rank", "kv_rank", "rot_dim", "vdim"):
        with_config(lambda c: mixer(c, 1).pop(key))
    with_config(lambda c: mixer(c, 1).update(q_rank=0))
    with_config(lambda c: mixer(c, 2).pop("right"))
    with_config(lambda c: mixer(c, 2).pop("left"))
    with_config(lambda c: mixer(c, 2)["right"].update(width=0))
    with_config(lambda c: c["layers"][0].update(type="latent_attention_2"))
    with_config(lambda c: c["layers"][0].update(mlp={"kind": "dense", "ff": 8}))
    with_config(lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3))
    with_config(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))           # more than the kept groups hold


def test_heads_that_may_mix_their_scores(pkg):
    assert 96 <= pkg.lib.cmlb200_talk_scores_heads() < 999


def test_tensor_file_refusals(pkg, synth, tmp_path):
    cfg, w, folder = lm_util.build(synth, tmp_path, "plain")
    path = folder / "model.safetensors"
    raw = path.read_bytes()
    n = int.from_bytes(raw[:8], "little")
    head = json.loads(raw[8:8 + n])

    def with_header(change):
        h = json.loads(json.dumps(head))
        change(h)
        t = json.dumps(h).encode()
        path.write_bytes(len(t).to_bytes(8, "little") + t + raw[8 + n:])
        assert not _load(pkg, folder)

    with_header(lambda h: h.pop("embed"))
    with_header(lambda h: h["embed"].update(dtype="U8"))
    with_header(lambda h: h["embed"].update(shape=[64, 63]))
    with_header(lambda h: h["embed"].update(data_offsets=[0, 1 << 40]))
    with_header(lambda h: h["embed"].update(data_offsets=[8, 4]))
    for bad in (b"", raw[:4], (1 << 60).to_bytes(8, "little") + raw[8:], raw[:8 + n // 2]):
        path.write_bytes(bad)
        assert not _load(pkg, folder)


def test_which_latents_run_on_the_tensor_cores(pkg):
    """Usual sizes do; a pool of unknown extent and what exceeds shared memory go to the other form."""
    def fits(rank, rot, pool_blocks=8):
        a = pkg.Latent(heads=16, dim=64, rot_dim=rot, vdim=64, rank=rank, ld=(rank + rot + 15) // 16 * 16, ld_rank=(rank + 63) // 64 * 64, pool_blocks=pool_blocks)
        return pkg.lib.cmlb200_attention_latent_tc_fits(a)
    for rank, rot in ((512, 64), (512, 32), (256, 64), (300, 64), (128, 128), (16, 2), (72, 24)):
        assert fits(rank, rot) == 1
    assert fits(512, 64, 0) == 0 and fits(512, 128) == 0 and fits(513, 16) == 0
    assert pkg.lib.cmlb200_attention_latent_tc_fits(None) == 0
    assert pkg.lib.cmlb200_set_attention_latent_form(3) == -1 and pkg.lib.cmlb200_set_attention_latent_form(0) == 0


def test_null_arguments(pkg):
    lib = pkg.lib
    lib.cml_lm_free(None)
    assert not lib.cml_lm_load(None, None) and lib.cml_lm_sequence_open(None) == -1 and lib.cml_lm_sequence_close(None, 0) == -1
    assert lib.cml_lm_step(None, None, 0, None) == -1 and lib.cml_lm_step_greedy(None, None, 0, None) == -1
    assert lib.cml_serving_run_lm(None, None, None, 0, None, None) == -1 and not lib.cml_lm_generate(None, None, 0, None)


# ---- blocks ----------------------------------------------------------------------------------------------
def test_blocks_are_taken_released_and_used_again(pkg):
    lib = pkg.lib
    c = lib.cml_paged_kv_cache_create_device(6, 3, 16)
    a, b = lib.cml_paged_cache_init_sequence(c), lib.cml_paged_cache_init_sequence(c)
    assert lib.cml_paged_cache_blocks_for(c, a, 16) == 1 and lib.cml_paged_cache_blocks_for(c, a, 17) == 2
    assert lib.cml_paged_cache_extend(c, a, 40) == 0 and c.contents.free_count == 3
    assert lib.cml_paged_cache_blocks_for(c, a, 8) == 0 and lib.cml_paged_cache_blocks_for(c, a, 9) == 1
    assert lib.cml_paged_cache_extend(c, b, 49) == -1 and c.contents.free_count == 3 and c.contents.sequences[b].seq_len == 0
    assert lib.cml_paged_cache_extend(c, b, 48) == 0 and c.contents.free_count == 0
    first = [c.contents.sequences[a].block_ids[i] for i in range(3)]
    lib.cml_paged_cache_release_before(c, a, 31)                       # block 1 still holds position 31
    assert c.contents.free_count == 1 and [c.contents.sequences[a].block_ids[i] for i in range(3)] == [-1] + first[1:]
    lib.cml_paged_cache_release_before(c, a, 32)
    lib.cml_paged_cache_release_before(c, a, -5)
    assert c.contents.free_count == 2
    assert lib.cml_paged_cache_extend(c, b, 17) == 0
    assert {c.contents.sequences[b].block_ids[i] for i in (3, 4)} == set(first[:2])
    lib.cml_paged_cache_free_sequence(c, a)
    lib.cml_paged_cache_free_sequence(c, b)
    assert c.contents.free_count == 6
    s = lib.cml_paged_cache_init_sequence(c)
    assert lib.cml_paged_cache_extend(c, s, 90) == 0 and c.contents.free_count == 0
    lib.cml_paged_cache_release_between(c, s, 17, 70)                  # blocks 0 and 1 hold the first 17 tokens, block 4 position 70
    kept = [c.contents.sequences[s].block_ids[i] >= 0 for i in range(6)]
    assert kept == [True, True, False, False, True, True] and c.contents.free_count == 2
    lib.cml_paged_cache_release_between(c, s, 17, 80)
    lib.cml_paged_cache_release_between(c, s, 17, 200)
    assert c.contents.free_count == 4
    lib.cml_paged_cache_free_sequence(c, s)
    assert c.contents.free_count == 6
    one = np.zeros(4, np.float32)
    s = lib.cml_paged_cache_init_sequence(c)
    assert lib.cml_paged_cache_append(c, s, pkg.np_ptr(one), pkg.np_ptr(one)) == -1          # no host data
    lib.cml_paged_kv_cache_free(c)
    assert not lib.cml_paged_kv_cache_create_device(0, 1, 16)


# ---- programs --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["trace_run", "cml_generate"])
def test_programs_build_and_refuse_bad_arguments(name):
    run = lambda *a: subprocess.run([str(ROOT / "bin" / name), *a], capture_output=True, text=True, timeout=600)
    r = run()
    assert r.returncode == 2 and "usage" in r.stderr
    r = run("--nonsense", "1")
    assert r.returncode == 2 and "unknown option" in r.stderr
    args = ["--model", "/nonexistent"] + (["--out", "/tmp", "--max-tokens", "64"] if name == "trace_run" else ["--tokens", "1,2"])
    r = run(*args)
    assert r.returncode == 2 and "cannot load" in r.stderr
