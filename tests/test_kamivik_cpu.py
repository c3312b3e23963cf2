"""CPU: the float64 Kamivik oracle against closed forms written out by hand, its own state handling under portions, and the
configuration reader key by key.  The engine is compared with this oracle in tests/test_kamivik_gpu.py."""
import copy
import math

import numpy as np
import pytest

from helix_b200 import engine as E
from helix_b200 import weights_io
from oracle import kamivik_ref as ref


def rnd(seed, *shape):
    return np.random.default_rng(seed).standard_normal(shape)


def test_norm_has_eps_inside_the_root_and_a_plain_gain():
    x, w = rnd(0, 3, 7) * 1e-3, rnd(1, 7)
    y = ref.rms_norm(x, w, 1e-5)
    for t in range(3):
        assert np.allclose(y[t], x[t] / math.sqrt(sum(v * v for v in x[t]) / 7 + 1e-5) * w)


def test_rotation_pairs_neighbours():
    x = rnd(2, 4, 3, 8)
    pos = np.array([0, 1, 9, 5000])
    y = ref.rotate_interleaved(x, pos, 50.0, 6)
    assert np.array_equal(y[..., 6:], x[..., 6:]) and np.allclose(y[0], x[0])
    for i in range(3):
        a = pos * 50.0 ** (-2.0 * i / 6)
        u, v = x[:, 2, 2 * i], x[:, 2, 2 * i + 1]
        assert np.allclose(y[:, 2, 2 * i], u * np.cos(a) - v * np.sin(a))
        assert np.allclose(y[:, 2, 2 * i + 1], v * np.cos(a) + u * np.sin(a))
    q, k = rnd(3, 1, 6), rnd(4, 1, 6)
    s = lambda a, b: float(ref.rotate_interleaved(q, [a], 50.0, 6)[0] @ ref.rotate_interleaved(k, [b], 50.0, 6)[0])
    assert abs(s(40, 33) - s(2007, 2000)) < 1e-9  # scores depend on the distance only


def test_window_edges_and_causality():
    pos = np.arange(10)
    full, win = ref.visible(pos, pos, None), ref.visible(pos, pos, 4)
    for i in range(10):
        assert [j for j in range(10) if full[i, j]] == list(range(i + 1))
        assert [j for j in range(10) if win[i, j]] == list(range(max(0, i - 3), i + 1))


@pytest.mark.parametrize("kind", [ref.FULL, ref.WIN])
def test_latent_attention_by_hand(kind):
    cfg = ref.random_config(order=((kind, False),), window=3)
    sd = ref.random_state_dict(cfg, 5)
    o = ref.KamivikOracle(cfg, sd)
    m, p = cfg["layers"][0]["mixer"], {k[7:]: v.astype(float) for k, v in sd.items() if k.startswith("l0.mix.")}
    h = rnd(6, 5, cfg["width"])
    got = o.mixer(0, cfg["layers"][0], h, o.new_state(), np.arange(5))
    H, Dk, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    turn = lambda v, t: ref.rotate_interleaved(v[None], [t], m["rot"]["base"], Dr)[0]
    t, heads = 4, []
    for hh in range(H):
        q = p["q"][hh * (Dk + Dr):(hh + 1) * (Dk + Dr)] @ h[t]
        s, vals = [], []
        for j in range(0 if kind == ref.FULL else t - 2, t + 1):
            d = p["dkv"] @ h[j]
            c = d[:R] / math.sqrt((d[:R] ** 2).mean() + 1e-5) * p["dkv.norm"]
            s.append((q[:Dk] @ (p["uk"][hh * Dk:(hh + 1) * Dk] @ c) + turn(q[Dk:], t) @ turn(d[R:], j)) * m["scale"])
            vals.append(p["uv"][hh * Dv:(hh + 1) * Dv] @ c)
        w = np.exp(s) / np.exp(s).sum()  # an ordinary softmax: no further term in the denominator
        out = (w[:, None] * np.array(vals)).sum(0)
        gate = ref.sigmoid(p["g"][hh] @ h[t]) if kind == ref.FULL else ref.sigmoid(p["g"][hh * Dv:(hh + 1) * Dv] @ h[t])
        heads.append(out * gate)
    assert np.allclose(got[t], p["o"] @ np.concatenate(heads))


def test_router_bias_joins_the_logits_and_weights_cover_the_chosen_only():
    h, W, b = rnd(7, 6, 9), rnd(8, 5, 9), rnd(9, 5)
    ids, w = ref.route(h, W, b, 2)
    for t in range(6):
        z = W @ h[t] + b
        assert list(ids[t]) == list(np.argsort(-z)[:2])
        e = np.exp(z[ids[t]])
        assert np.allclose(w[t], e / e.sum())
    assert any(list(ids[t]) != list(np.argsort(-(W @ h[t]))[:2]) for t in range(6))  # the bias changes choices
    assert np.allclose(ref.route(h, W, b, 1)[1], 1.0)
    assert np.all(np.isinf(ref.route_margin(h, W, b, 5)))


def test_experts_are_ungated_erf_gelu_units():
    h, up, down = rnd(10, 4, 6), rnd(11, 8, 6), rnd(12, 6, 8)
    z = h @ up.T
    act = np.array([[0.5 * v * (1 + math.erf(v / math.sqrt(2))) for v in row] for row in z])
    assert np.allclose(ref.expert(h, up, down), act @ down.T)
    p = {"router": rnd(13, 3, 6), "router.b": rnd(14, 3)}
    for e in range(3):
        p[f"e{e}.up"], p[f"e{e}.down"] = rnd(20 + e, 8, 6), rnd(30 + e, 6, 8)
    y = ref.mixture(h, p, dict(router=dict(experts=3, top=2)))
    ids, w = ref.route(h, p["router"], p["router.b"], 2)
    for t in range(4):
        assert np.allclose(y[t], sum(w[t, k] * ref.expert(h[t:t + 1], p[f"e{ids[t, k]}.up"], p[f"e{ids[t, k]}.down"])[0] for k in range(2)))


def test_layer_adds_both_sublayers_of_one_norm():
    cfg = ref.random_config(order=((ref.WIN, True),), mult=0.3)
    sd = ref.random_state_dict(cfg, 7)
    o = ref.KamivikOracle(cfg, sd)
    toks = [3, 5, 8]
    taps = []
    logits = o.forward(toks, taps=taps)
    x = sd["embed"][toks].astype(float)
    h = ref.rms_norm(x, sd["l0.norm1"], 1e-5)
    a = o.mixer(0, cfg["layers"][0], h, o.new_state(), np.arange(3))
    f = ref.mixture(h, o.sub("l0.mlp."), cfg["layers"][0]["mlp"])
    y = x + 0.3 * (sd["l0.ls1"] * a + sd["l0.ls2"] * f)
    assert np.allclose(taps[0], y)
    assert np.allclose(logits, ref.rms_norm(y, sd["final.norm"], 1e-5) @ sd["head"].T.astype(float))


def test_portions_continue_from_the_kept_rows():
    cfg = ref.random_config()
    o = ref.KamivikOracle(cfg, ref.random_state_dict(cfg, 1))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60)
    whole = o.forward(toks)
    for cuts in ([2] * 30, [1] * 60, [37, 23], [36, 1, 2, 21]):
        st, out, at = o.new_state(), [], 0
        for n in cuts:
            out.append(o.forward(toks[at:at + n], st))
            at += n
        assert np.allclose(np.concatenate(out), whole)


def test_choices_of_the_random_checkpoints_are_clear():
    for kw in (dict(), dict(experts=70, top=5, width=160), dict(experts=24, top=4, width=128)):
        cfg = ref.random_config(**kw)
        margins = []
        ref.KamivikOracle(cfg, ref.random_state_dict(cfg, 3)).forward(np.arange(100) % cfg["vocab"], margins=margins)
        assert np.min(margins) > 0.3


def test_configuration_reader():
    cfg = ref.random_config(per_layer={2: ref.mixer_cfg(heads=5, dim=40, rot_dim=24, vdim=56, kv_rank=72, base=77.0, scale=0.123)}, mult=0.6, eps=3e-6)
    d = weights_io.desc_from_hf_config(copy.deepcopy(cfg), compute_f32=True)
    assert (d.width, d.vocab, d.compute_f32, len(d.layers)) == (96, 120, 1, 3)
    assert (d.norm_place, d.norm_kind, d.one_norm, d.layer_scale, d.plain_gains, d.embed_norm, d.tie_head) == (E.NORM_PARALLEL, E.NORM_RMS, 1, 1, 1, 0, 0)
    assert d.norm_eps == 3e-6 and d.resid_mult == 0.6 and d.logit_softcap == 0.0 and d.logit_scale in (0.0, 1.0)
    a, b, c = d.layers
    assert (a.mixer, a.mask, a.attn_flags) == (E.MIXER_LATENT, E.MASK_CAUSAL, E.ATTN_NO_SINK | E.ATTN_HEAD_GATE)
    assert (b.mixer, b.mask, b.window, b.attn_flags) == (E.MIXER_LATENT, E.MASK_WINDOW, 37, E.ATTN_NO_SINK)
    assert (c.heads, c.dim, c.rot_dim, c.rope_dims, c.vdim, c.kv_rank, c.q_rank, c.rope_base, c.rope_pairing) == (5, 40, 24, 24, 56, 72, 0, 77.0, 1)
    assert c.scale == 0.123 and c.ff == 0 and c.kv_from == -1
    assert (a.ff_kind, a.ff, a.experts, a.top_k, a.identity_experts) == (E.FF_MOE, 40, 6, 2, 0)
    assert (a.router_kind, a.expert_kind, a.route_bias, a.shared_ff) == (E.ROUTER_CHOSEN, E.EXPERT_GELU, 1, 0)
    assert d.unused_tensors == {"l2.ls2"}
    for edit in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                 lambda c: c.update(residual_mult=0.0)):
        bad = copy.deepcopy(cfg)
        edit(bad)
        with pytest.raises(ValueError):
            weights_io.desc_from_hf_config(bad)
