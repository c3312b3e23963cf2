"""CPU: the float64 Pupalix oracle against closed forms written out by hand, its own state handling under portions, and the
configuration reader key by key.  The engine is compared with this oracle in tests/test_pupalix_gpu.py."""
import copy
import ctypes as C
import math

import numpy as np
import pytest

from helix_b200 import engine as E
from helix_b200 import weights_io
from oracle import pupalix_ref as ref
from oracle.pupalix_ref import GQA, LATENT, LIGHT


def rnd(seed, *shape):
    return np.random.default_rng(seed).standard_normal(shape)


def test_norm_has_eps_inside_the_root_and_a_plain_gain():
    x, w = rnd(0, 3, 7) * 1e-3, rnd(1, 7)
    y = ref.rms_norm(x, w, 1e-5)
    for t in range(3):
        assert np.allclose(y[t], x[t] / math.sqrt(sum(v * v for v in x[t]) / 7 + 1e-5) * w)


def test_embedding_adds_the_row_of_the_pair():
    table, big = rnd(2, 9, 4), rnd(3, 6, 4)  # five buckets and the row of a first token
    y = ref.embed([4, 8, 0], None, table, big, 3.0, 7, 2)
    assert np.allclose(y[0], 3.0 * table[4] + big[5])
    assert np.allclose(y[1], 3.0 * table[8] + big[(4 * 7 + 8 * 2) % 5])
    assert np.allclose(y[2], 3.0 * table[0] + big[(8 * 7 + 0 * 2) % 5])
    assert np.allclose(ref.embed([8, 0], 4, table, big, 3.0, 7, 2), y[1:])


def test_streams_are_mixed_from_the_old_ones():
    xs, y, mix, out, w = rnd(4, 3, 2, 5), rnd(5, 2, 5), rnd(6, 3, 3), rnd(7, 3), rnd(8, 3)
    new = ref.write_streams(xs, y, mix, out)
    for t in range(3):
        assert np.allclose(new[t], sum(mix[s, t] * xs[s] for s in range(3)) + out[t] * y)
    assert np.allclose(ref.read_streams(xs, w), w[0] * xs[0] + w[1] * xs[1] + w[2] * xs[2])


def test_rotation_pairs_neighbours_and_is_scaled_per_frequency():
    x, pos = rnd(9, 4, 3, 8), np.array([0, 1, 9, 5000])
    y = ref.rotate(x, pos, dict(dims=6, base=50.0))
    assert np.array_equal(y[..., 6:], x[..., 6:]) and np.allclose(y[0], x[0])
    for i in range(3):
        a = pos * 50.0 ** (-2.0 * i / 6)
        u, v = x[:, 2, 2 * i], x[:, 2, 2 * i + 1]
        assert np.allclose(y[:, 2, 2 * i], u * np.cos(a) - v * np.sin(a))
        assert np.allclose(y[:, 2, 2 * i + 1], v * np.cos(a) + u * np.sin(a))
    sc = dict(factor=4.0, original=100, fast=6.0, slow=1.0)
    f, mult = ref.yarn(16, 100.0, sc)
    plain = 100.0 ** (-2.0 * np.arange(8) / 16)
    assert math.isclose(mult, 0.1 * math.log(4.0) + 1.0)
    lo = math.floor(16 * math.log(100 / (2 * math.pi * 6.0)) / (2 * math.log(100.0)))
    hi = math.ceil(16 * math.log(100 / (2 * math.pi * 1.0)) / (2 * math.log(100.0)))
    assert 0 < lo < hi < 8
    for i in range(8):
        r = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        assert math.isclose(f[i], plain[i] * (r / 4.0 + 1.0 - r))
    assert f[0] == plain[0] and math.isclose(f[7], plain[7] / 4.0)
    z = ref.rotate(x, pos, dict(dims=8, base=100.0, scaling=sc))
    assert np.allclose(z[0], x[0] * mult)  # cos and sin carry the factor at every position
    # a bend that lies before the first frequency, and one narrower than the ramp's least width
    assert np.allclose(ref.yarn(8, 100.0, dict(factor=2.0, original=5, fast=32.0, slow=1.0))[0][1:], 100.0 ** (-2.0 * np.arange(1, 4) / 8) / 2.0)


def test_blocks_are_counted_from_position_zero():
    pos = np.arange(3, 10)
    seen = ref.visible(pos, np.arange(10), 4)
    for i, p in enumerate(pos):
        assert [j for j in range(10) if seen[i, j]] == list(range(p // 4 * 4, p + 1))
    assert ref.visible(pos, np.arange(10), None).sum() == sum(p + 1 for p in pos)


@pytest.mark.parametrize("kind", [LATENT, GQA])
def test_attention_by_hand(kind):
    cfg = ref.random_config(order=((kind, None),), gqa=ref.gqa_cfg(block=3, softcap=2.0), loop=None)
    sd = ref.random_state_dict(cfg, 5)
    o = ref.PupalixOracle(cfg, sd)
    m, p = cfg["layers"][0]["mixer"], {k[7:]: v.astype(float) for k, v in sd.items() if k.startswith("l0.mix.")}
    h = rnd(6, 5, cfg["width"])
    got = o.mixer(0, 0, h, o.new_state(), np.arange(5))
    H, Dk, Dv, t, heads = m["heads"], m["dim"], m["vdim"], 4, []
    turn = lambda v, at: ref.rotate(v[None], [at], m["rot"])[0]
    nrm = lambda v, w: v / math.sqrt((v ** 2).mean() + 1e-5) * w
    for hh in range(H):
        s, vals = [], []
        if kind == LATENT:
            Dr, R = m["rot_dim"], m["kv_rank"]
            q = p["q"][hh * (Dk + Dr):(hh + 1) * (Dk + Dr)] @ h[t]
            for j in range(t + 1):
                d = p["dkv"] @ h[j]
                c = nrm(d[:R], p["dkv.norm"])
                s.append((q[:Dk] @ (p["uk"][hh * Dk:(hh + 1) * Dk] @ c) + turn(q[Dk:], t) @ turn(d[R:], j)) * m["scale"])
                vals.append(p["uv"][hh * Dv:(hh + 1) * Dv] @ c)
        else:
            g = hh // (H // m["kv_heads"])
            q = nrm(p["q"] @ h[t], p["q.norm"])[hh * Dk:(hh + 1) * Dk]
            for j in range(3, t + 1):  # position 4 lies in the block 3 .. 5
                k = p["k"] @ h[j]
                s.append(2.0 * math.tanh(q @ nrm(k, p["k.norm"])[g * Dk:(g + 1) * Dk] * m["scale"] / 2.0))
                vals.append(k[g * Dk:(g + 1) * Dk])  # the projection itself
        w = np.exp(s) / np.exp(s).sum()
        heads.append((w[:, None] * np.array(vals)).sum(0))
    assert np.allclose(got[t], p["o"] @ np.concatenate(heads))


def test_linear_attention_by_hand():
    cfg = ref.random_config(order=((LIGHT, None),), loop=None)
    sd = ref.random_state_dict(cfg, 5)
    o = ref.PupalixOracle(cfg, sd)
    m, p = cfg["layers"][0]["mixer"], {k[7:]: v.astype(float) for k, v in sd.items() if k.startswith("l0.mix.")}
    h = rnd(6, 4, cfg["width"])
    got = o.mixer(0, 0, h, o.new_state(), np.arange(4))
    silu = lambda z: z / (1 + np.exp(-z))
    t, heads = 3, []
    for hh, a in enumerate(m["decay"]):
        row = lambda n, d, j: silu(p[n][hh * d:(hh + 1) * d] @ h[j])
        heads.append(sum(a ** (t - j) * (row("q", m["dim"], t) @ row("k", m["dim"], j)) * row("v", m["vdim"], j) for j in range(4)))
    y = np.concatenate(heads)
    y = y / math.sqrt((y ** 2).mean() + 1e-5) * p["norm"] / (1 + np.exp(-(p["g"] @ h[t])))
    assert np.allclose(got[t], p["o"] @ y)


def test_router_scores_all_experts_and_ranks_groups_by_their_largest():
    h, W = rnd(10, 40, 9), rnd(11, 12, 9)
    r = dict(experts=12, top=3, groups=dict(count=4, keep=2))
    ids, w = ref.route(h, W, r)
    differs = 0
    for t in range(40):
        z = W @ h[t]
        s = np.exp(z) / np.exp(z).sum()
        best = sorted(range(4), key=lambda g: -max(s[3 * g:3 * g + 3]))[:2]
        want = sorted([e for e in range(12) if e // 3 in best], key=lambda e: -s[e])[:3]
        assert list(ids[t]) == want and np.allclose(w[t], s[want])  # softmax over all twelve, not renormalised
        pair = sorted(range(4), key=lambda g: -np.sort(s[3 * g:3 * g + 3])[-2:].sum())[:2]
        differs += sorted(pair) != sorted(best)
    assert differs > 0
    ids, w = ref.route(h, W, dict(experts=12, top=3))
    assert all(list(ids[t]) == list(np.argsort(-(W @ h[t]))[:3]) for t in range(40))


def test_feed_forward_units():
    h, gate, up, down = rnd(12, 4, 6), rnd(13, 8, 6), rnd(14, 8, 6), rnd(15, 6, 8)
    g, u = h @ gate.T, h @ up.T
    assert np.allclose(ref.expert(h, gate, up, down), (g / (1 + np.exp(-g)) * u) @ down.T)
    act = 0.5 * g * (1 + np.tanh(math.sqrt(2 / math.pi) * (g + 0.044715 * g ** 3)))
    assert np.allclose(ref.dense(h, dict(gate=gate, up=up, down=down)), (act * u) @ down.T)


def test_loop_order_and_state_of_each_pass():
    cfg = ref.random_config(loop=(1, 3, 3))
    assert ref.runs(cfg) == [0, 1, 2, 1, 2, 1, 2, 3]
    assert ref.runs(ref.random_config(loop=None)) == [0, 1, 2, 3]
    o = ref.PupalixOracle(cfg, ref.random_state_dict(cfg, 3))
    st, taps = o.new_state(), []
    o.forward([1, 2, 3], st, taps=taps)
    assert sorted(st["rows"]) == list(range(8)) and len(taps) == 8
    assert not np.allclose(st["rows"][1][0], st["rows"][3][0])


def test_layer_and_output_by_hand():
    cfg = ref.random_config(order=((LIGHT, "dense"),), loop=None, streams=2)
    sd = ref.random_state_dict(cfg, 7)
    o = ref.PupalixOracle(cfg, sd)
    toks, taps = [3, 5, 8], []
    logits = o.forward(toks, taps=taps)
    s = {k: v.astype(float) for k, v in sd.items()}
    b = cfg["embedding"]["bigram"]
    x = ref.embed(toks, None, s["embed"], s["bigram"], cfg["embedding"]["scale"], b["mul_prev"], b["mul_cur"])
    x1, x2 = x, x
    for q, f in ((1, lambda h: o.mixer(0, 0, h, o.new_state(), np.arange(3))), (2, lambda h: ref.dense(h, o.sub("l0.mlp.")))):
        i, ou, mx = s[f"l0.hc{q}.in"], s[f"l0.hc{q}.out"], s[f"l0.hc{q}.mix"]
        y = f(ref.rms_norm(i[0] * x1 + i[1] * x2, s[f"l0.norm{q}"], 1e-5))
        x1, x2 = mx[0, 0] * x1 + mx[1, 0] * x2 + ou[0] * y, mx[0, 1] * x1 + mx[1, 1] * x2 + ou[1] * y
    assert np.allclose(taps[0], x1 + x2)
    z = ref.rms_norm(x1 + x2, s["final.norm"], 1e-5) @ s["embed"].T * cfg["logit_scale"]
    assert np.allclose(logits, cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"]))


def test_portions_continue_from_the_kept_state():
    cfg = ref.random_config()
    o = ref.PupalixOracle(cfg, ref.random_state_dict(cfg, 1))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60)
    whole = o.forward(toks)
    for cuts in ([2] * 30, [1] * 60, [37, 23], [36, 1, 2, 21]):
        st, out, at = o.new_state(), [], 0
        for n in cuts:
            out.append(o.forward(toks[at:at + n], st))
            at += n
        assert np.allclose(np.concatenate(out), whole)


def test_choices_of_the_random_checkpoints_are_clear():
    for kw in (dict(), dict(moe=ref.moe_cfg(70, 5, 24, None), width=160), dict(moe=ref.moe_cfg(24, 4, 40, (6, 3)), width=128), dict(streams=5)):
        cfg = ref.random_config(**kw)
        margins = []
        ref.PupalixOracle(cfg, ref.random_state_dict(cfg, 3)).forward(np.arange(100) % cfg["vocab"], margins=margins)
        assert np.min(margins) > 0.3


def test_configuration_reader():
    cfg = ref.random_config(per_layer={1: ref.latent_cfg(heads=5, dim=40, rot_dim=24, vdim=56, kv_rank=72, base=77.0, scale=0.123)},
                            per_mlp={3: None}, eps=3e-6, mul=(200, 5))
    d = weights_io.desc_from_hf_config(copy.deepcopy(cfg), compute_f32=True)
    assert (d.width, d.vocab, d.compute_f32, len(d.layers)) == (96, 120, 1, 4)
    assert (d.norm_place, d.norm_kind, d.streams, d.plain_gains, d.embed_norm, d.tie_head) == (E.NORM_PRE, E.NORM_RMS, 3, 1, 0, 1)
    assert (d.norm_eps, d.embed_scale, d.logit_scale, d.logit_softcap) == (3e-6, 2.5, 0.5, 12.0)
    assert (d.bigram_buckets, d.bigram_mul_prev, d.bigram_mul_cur) == (97, 200 % 97, 5)
    assert (d.loop_start, d.loop_stop, d.loop_times) == (1, 3, 2)
    a, b, c, e = d.layers
    assert (a.mixer, a.heads, a.dim, a.vdim, a.head_decay) == (E.MIXER_LIGHTNING, 3, 24, 40, (0.5, 0.93, 0.998))
    assert (a.ff_kind, a.ff) == (E.FF_GELU_TANH, 72)
    assert (b.mixer, b.mask, b.attn_flags, b.rope_pairing) == (E.MIXER_LATENT, E.MASK_CAUSAL, E.ATTN_NO_SINK | E.ATTN_NO_GATE, 1)
    assert (b.heads, b.dim, b.rot_dim, b.rope_dims, b.vdim, b.kv_rank, b.q_rank, b.rope_base, b.scale) == (5, 40, 24, 24, 56, 72, 0, 77.0, 0.123)
    assert (b.rope_yarn_factor, b.rope_original, b.rope_yarn_fast, b.rope_yarn_slow) == (4.0, 60, 8.0, 1.0)
    assert (b.ff_kind, b.ff, b.experts, b.top_k, b.route_groups, b.route_keep, b.route_group_max, b.route_plain) == (E.FF_MOE, 40, 6, 3, 3, 2, 1, 1)
    assert (b.router_kind, b.expert_kind, b.route_renorm, b.route_bias, b.shared_ff) == (E.ROUTER_SOFTMAX, E.EXPERT_SILU, 0, 0, 0)
    assert (c.mixer, c.mask, c.window, c.attn_flags, c.score_cap) == (E.MIXER_GQA, E.MASK_CHUNK, 37, E.ATTN_V_IS_K | E.ATTN_QK_PROJ_NORM, 20.0)
    assert (c.heads, c.kv_heads, c.dim, c.vdim, c.rope_dims) == (4, 2, 24, 24, 0)
    assert e.ff == 0 and d.unused_tensors == {"l3.norm2", "l3.hc2.in", "l3.hc2.out", "l3.hc2.mix"}
    # what a configuration may leave out
    less = copy.deepcopy(cfg)
    for k in ("loop", "logit_softcap", "logit_scale"):
        less.pop(k)
    less["streams"] = 1
    del less["layers"][1]["mixer"]["rot"]["scaling"], less["layers"][1]["mlp"]["router"]["groups"]
    del less["layers"][2]["mixer"]["mask"], less["layers"][2]["mixer"]["softcap"]
    d = weights_io.desc_from_hf_config(less)
    assert d.loop_times == 0 and d.logit_softcap == 0.0 and d.logit_scale == 1.0 and d.streams == 1
    assert d.layers[1].rope_yarn_factor == 0.0 and d.layers[1].route_groups == 0
    assert d.layers[2].mask == E.MASK_CAUSAL and d.layers[2].score_cap == 0.0
    assert weights_io.desc_from_hf_config(less, shapes={"l0.norm1": (96,)}).streams == 0  # no read / write weights: one plain stream
    for edit in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c.update(logit_scale=0.0),
                 lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), lambda c: c["loop"].update(times=0)):
        bad = copy.deepcopy(cfg)
        edit(bad)
        with pytest.raises(ValueError):
            weights_io.desc_from_hf_config(bad)


def test_descriptions_carry_the_decays():
    layers = [E.LayerDesc(mixer=E.MIXER_LIGHTNING, heads=2, head_decay=(0.5, i / 64.0)) for i in range(50)] + [E.LayerDesc()]
    _, arr = E.StackDesc(layers=layers).to_c()
    junk = [(C.c_float * 2)(7.0, 7.0) for _ in range(200)]
    assert all(arr[i].head_decay[0] == 0.5 and arr[i].head_decay[1] == i / 64.0 for i in range(50)) and not arr[50].head_decay
    assert len(junk) == 200
