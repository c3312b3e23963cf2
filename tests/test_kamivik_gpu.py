"""Kamivik layer-list decoders through the engine (driven sequences and the scheduler) against the float64 oracle.

Every test builds its own small configuration and random bf16-representable weights (oracle/kamivik_ref.py; router choices are
made clear there, so no comparison rests on a close call); the engine runs them in its exact mode (fp32 weights, cache and
products), where a key left out, a window off by one or a wrong gate must show, and in its serving mode (bf16 weights / cache
rows / GEMM operands; long portions on the fused attention over expanded rows, single tokens and short portions on the
latent-row kernel, other shapes on the per-token kernel) with a rounding-sized bound.
"""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import helix_b200 as hb
from helix_b200 import weights_io
from helix_b200.engine import CAPTURE_PROMPT_LOGITS, CAPTURE_STEP_LOGITS
from oracle import kamivik_ref as ref
from oracle.kamivik_ref import FULL, WIN, mixer_cfg

pytestmark = pytest.mark.gpu

TOL = {1: 2e-4, 0: 6e-2}  # compute_f32 -> bound on rms(diff) / rms(expected) per logits row


def row_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean(-1))


def make_engine(cfg, sd, f32, max_seqs=4, ctx=512, pool=0, batched=0, edit=None, **kw):
    desc = weights_io.desc_from_hf_config(copy.deepcopy(cfg), {k: v.shape for k, v in sd.items()}, compute_f32=bool(f32))
    if edit:
        edit(desc)
    e = hb.Engine(hb.EngineConfig(device=0, max_seqs=max_seqs, max_ctx=ctx, max_batched_tokens=batched or ctx, kv_pool_tokens=pool, **kw))
    e.load_state_dict(desc, sd)
    return e


def tokens(seed, n, vocab):
    return np.random.default_rng(seed).integers(0, vocab - 1, n).tolist()  # vocab - 1 is the marker of plant_marker


def replay(e, toks, cuts):
    """Feed one sequence in portions of the given sizes (the rest one token at a time), all positions wanted."""
    sid, out, at = e.seq_open(), [], 0
    cuts = list(cuts)
    while at < len(toks):
        n = min(cuts.pop(0) if cuts else 1, len(toks) - at)
        out.append(e.seq_step([(sid, toks[at:at + n], list(range(n)))]))
        at += n
    e.seq_close(sid)
    return np.concatenate(out)


CONFIGS = {
    "default": dict(),
    "causal_alone": dict(order=((FULL, False),)),
    "window_alone": dict(order=((WIN, False),)),
    "experts_on_causal": dict(order=((FULL, True),)),
    "experts_on_window": dict(order=((WIN, True),)),
    "one_head": dict(full=mixer_cfg(heads=1, dim=64, rot_dim=16, vdim=72, kv_rank=64), win=mixer_cfg(heads=1, dim=48, rot_dim=48, vdim=64, kv_rank=24)),
    "seventeen_heads": dict(full=mixer_cfg(heads=17, dim=8, rot_dim=8, vdim=8, kv_rank=32), win=mixer_cfg(heads=33, dim=16, rot_dim=8, vdim=8, kv_rank=72)),
    # nothing a multiple of 8: every product takes the CUDA-core GEMM, attention the per-token kernel
    "odd_sizes": dict(width=90, vocab=131, ff=50, full=mixer_cfg(heads=5, dim=9, rot_dim=6, vdim=7, kv_rank=22), win=mixer_cfg(heads=3, dim=11, rot_dim=2, vdim=13, kv_rank=35)),
    # values a model may make equal or one
    "equal_sizes": dict(full=mixer_cfg(heads=2, dim=32, rot_dim=32, vdim=32, kv_rank=32), win=mixer_cfg(heads=2, dim=32, rot_dim=32, vdim=32, kv_rank=32, base=1000.0)),
    "neutral_constants": dict(mult=1.0, full=mixer_cfg(scale=1.0), win=mixer_cfg(scale=1.0), experts=1, top=1),
    "every_expert_chosen": dict(experts=3, top=3),
    "one_of_many": dict(experts=9, top=1),
    "many_experts": dict(experts=70, top=5, width=160, ff=24),  # router wider than one MMA tile
    "ten_of_twenty": dict(experts=20, top=10, width=128),       # more expert rows per token than the residual step keeps in registers
    "window_of_one": dict(window=1),
    "window_of_two": dict(window=2),
    "window_of_a_page": dict(window=64),
    "window_beyond_the_prompt": dict(window=400),
    "layers_differ": dict(order=((WIN, True), (FULL, False), (FULL, True), (WIN, False)),
                          per_layer={2: mixer_cfg(heads=2, dim=40, rot_dim=24, vdim=56, kv_rank=104, base=50.0, scale=0.3),
                                     3: dict(mixer_cfg(heads=6, dim=16, rot_dim=8, vdim=16, kv_rank=16), mask=dict(size=90))},
                          per_mlp={2: dict(kind="moe", expert=dict(ff=64), router=dict(experts=4, top=3))}),
    # every sub-tile count of the two tensor-core attention kernels: unrotated parts up to 128, values up to 128, latents up to 512
    "wide_heads": dict(width=128, ff=64, full=mixer_cfg(heads=3, dim=128, rot_dim=64, vdim=128, kv_rank=512), win=mixer_cfg(heads=2, dim=72, rot_dim=40, vdim=64, kv_rank=136)),
    "middling_heads": dict(width=128, ff=64, full=mixer_cfg(heads=2, dim=64, rot_dim=64, vdim=104, kv_rank=320), win=mixer_cfg(heads=20, dim=48, rot_dim=16, vdim=40, kv_rank=256)),
    "beyond_the_kernels": dict(width=128, full=mixer_cfg(heads=2, dim=136, rot_dim=16, vdim=64, kv_rank=64), win=mixer_cfg(heads=2, dim=32, rot_dim=72, vdim=136, kv_rank=520)),
}


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_portions_match_oracle(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=3)
    toks = tokens(1, 150, cfg["vocab"])  # crosses two page borders
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, f32) as e:
        assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[f32]
        assert row_err(replay(e, toks, [97, 2, 50]), want).max() < TOL[f32]


@pytest.mark.parametrize("name", ["default", "layers_differ", "wide_heads", "middling_heads", "many_experts", "ten_of_twenty"])
def test_steps_of_hundreds_of_tokens(name):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=5)
    toks = tokens(2, 430, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[f32]
            assert row_err(replay(e, toks, [300, 2, 97, 2]), want).max() < TOL[f32]


@pytest.mark.parametrize("name,f32", [("default", 1), ("default", 0), ("wide_heads", 0), ("odd_sizes", 0)])
def test_prefill_portions_and_single_tokens_agree(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=7)
    toks = tokens(3, 140, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, f32) as e:
        whole = replay(e, toks, [len(toks)])
        for cuts in ([64, 64], [63, 2, 2, 61], [19, 20, 21, 2, 45], [1, 1, 1, 2, 3, 64, 5], [2, 2, 2, 3, 2], []):
            got = replay(e, toks, cuts)
            assert row_err(got, want).max() < TOL[f32], cuts
            assert row_err(got, whole).max() < (1e-5 if f32 else 3e-2), cuts  # the same positions, cut differently: rounding only


def with_window(cfg, i, size):
    c = copy.deepcopy(cfg)
    c["layers"][i]["mixer"]["mask"] = dict(size=size)
    return c


@pytest.mark.parametrize("window,at", [(64, 0), (64, 1), (65, 63), (37, 27), (1, 70), (2, 62), (130, 5)])
def test_window_edges_in_prompts_and_in_decoding(window, at):
    # a marker token every head looks at while it is in the window: position at + window - 1 sees it, at + window does not
    cfg = ref.random_config(order=((WIN, True),), window=window)
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=11), [0])
    toks = tokens(4, at + window + 60, cfg["vocab"])
    toks[at] = cfg["vocab"] - 1
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    edge = at + window
    for size, row in ((window - 1, edge - 1), (window + 1, edge)):  # a window one off shows at exactly one of the two positions
        if size > 0:
            assert row_err(ref.KamivikOracle(with_window(cfg, 0, size), sd).forward(toks)[row:row + 1], want[row:row + 1])[0] > 3 * TOL[0]
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            # one prompt; decoding over the edge; portions that start or end on it; portions of two
            for cuts in ([len(toks)], [max(1, edge - 3)], [edge - 1, 2, 2, 2], [edge, 64], [2] * (len(toks) // 2 + 1), [max(1, edge - 66), 66, 2]):
                assert row_err(replay(e, toks, cuts), want).max() < TOL[f32], cuts


@pytest.mark.parametrize("name", ["default", "wide_heads", "odd_sizes"])
def test_far_keys_and_page_borders(name):
    # markers at the first token, at page borders and in between; the causal layer's queries hundreds of positions on still see them
    kw = dict(CONFIGS[name], order=((FULL, True), (FULL, False)))
    cfg = ref.random_config(**kw)
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=13), [0])
    for at in (0, 63, 64, 150):
        toks = tokens(5, 400, cfg["vocab"])
        o = ref.KamivikOracle(cfg, sd)
        plain = o.forward(toks)
        toks[at] = cfg["vocab"] - 1
        want = o.forward(toks)
        assert row_err(plain[-100:], want[-100:]).min() > 2 * TOL[0]  # what losing the far key would look like
        for f32 in (1, 0):
            with make_engine(cfg, sd, f32) as e:
                for cuts in ([len(toks)], [255, 2, 1, 1, 1, 2, 64], [64, 64, 128, 130]):
                    assert row_err(replay(e, toks, cuts), want).max() < TOL[f32], cuts


def test_keys_further_back_than_one_block_of_the_per_token_kernel():
    # exact mode, 4.5 thousand positions: the per-token kernel takes more than one block of keys; serving mode: many splits
    cfg = ref.random_config(order=((FULL, False),), full=mixer_cfg(heads=1, dim=16, rot_dim=8, vdim=72, kv_rank=24))
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=17), [0])
    toks = tokens(6, 4400, cfg["vocab"])
    toks[10] = toks[260] = cfg["vocab"] - 1
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32, ctx=4480, batched=2048) as e:
            sid, at, rows = e.seq_open(), 0, {}
            for n in (2048, 2048, 100, 2, 60, 1, 1, 1, 139):
                want_at = [n - 1] if n < 100 else [0, n // 2, n - 1]
                out = e.seq_step([(sid, toks[at:at + n], want_at)])
                for w, r in zip(want_at, out):
                    rows[at + w] = r
                at += n
            e.seq_close(sid)
            assert at == len(toks)
            idx = sorted(rows)
            assert row_err(np.stack([rows[i] for i in idx]), want[idx]).max() < TOL[f32]


def test_rotation_at_large_positions():
    # short wavelengths: positions in the hundreds turn many times, on the key part that all heads share and on the queries
    cfg = ref.random_config(order=((FULL, False), (WIN, False)), full=mixer_cfg(base=3.0, scale=0.3), win=mixer_cfg(base=2.0, rot_dim=16, scale=0.3), window=150)
    sd = ref.random_state_dict(cfg, seed=23)
    toks = tokens(8, 400, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    other = copy.deepcopy(cfg)
    other["layers"][0]["mixer"]["rot"]["base"] = 3.3
    assert row_err(ref.KamivikOracle(other, sd).forward(toks)[5:], want[5:]).max() > 50 * TOL[1]
    for f32, cuts in ((1, [len(toks)]), (1, [390]), (0, [199, 2]), (0, [len(toks)])):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, cuts), want).max() < TOL[f32]


def test_first_tokens_of_a_sequence():
    # an ordinary softmax: the first position has weight one on itself (a sink in the denominator would take a share of it)
    cfg = ref.random_config(order=((FULL, True), (WIN, True)))
    sd = ref.random_state_dict(cfg, seed=25)
    toks = tokens(9, 12, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32, max_seqs=1) as e:
            for cuts in ([], [1, 2, 2], [2, 3], [len(toks)]):
                assert row_err(replay(e, toks, cuts), want).max() < TOL[f32]


def test_gates_gains_factor_router_bias_and_activation_count():
    # where a plausible other reading exists the oracle states the design; the alternatives must differ, the engine follows the oracle
    cfg = ref.random_config(order=((FULL, True), (WIN, True)), mult=0.7)
    sd = ref.random_state_dict(cfg, seed=27)
    toks = tokens(10, 50, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)

    def alt(edit_cfg=None, **edit_sd):
        c, s = copy.deepcopy(cfg), dict(sd)
        if edit_cfg:
            edit_cfg(c)
        for k, f in edit_sd.items():
            for n in list(s):
                if n.endswith("." + k.replace("_", ".")):
                    s[n] = f(s[n])
        return ref.KamivikOracle(c, s).forward(toks)

    ones = lambda v: np.where(v == 0, 0, 1).astype(np.float32)
    for other in (alt(lambda c: c.update(residual_mult=1.0)), alt(ls1=ones), alt(ls2=ones), alt(router_b=np.zeros_like), alt(mix_g=np.zeros_like)):
        assert row_err(other, want).max() > 50 * TOL[1]
    act = ref.gelu_erf
    ref.gelu_erf = lambda z: 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
    try:
        assert row_err(ref.KamivikOracle(cfg, sd).forward(toks), want).max() > 1e-4  # the tanh form is another function
    finally:
        ref.gelu_erf = act
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, [33, 2]), want).max() < (5e-5 if f32 else TOL[0])


def test_long_decoding_over_pages():
    cfg = ref.random_config()
    sd = ref.random_state_dict(cfg, seed=31)
    toks = tokens(8, 230, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, 1) as e:
        assert row_err(replay(e, toks, [10]), want).max() < TOL[1]  # 220 single-token steps
    with make_engine(cfg, sd, 0, use_cuda_graphs=1) as e:
        assert row_err(replay(e, toks, [10]), want).max() < TOL[0]


@pytest.mark.parametrize("name,f32", [("default", 1), ("default", 0), ("wide_heads", 0), ("odd_sizes", 1), ("odd_sizes", 0)])
def test_mixed_batches_match_each_request_alone(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=33)
    o = ref.KamivikOracle(cfg, sd)
    seqs = [tokens(20 + i, n, cfg["vocab"]) for i, n in enumerate((150, 37, 90, 164))]
    want = [o.forward(s) for s in seqs]
    plans = [[64, 2, 30, 1, 1, 1, 51], [1, 1, 1, 1, 1, 1, 31], [3, 64, 2, 1, 20], [2, 2, 80, 2, 56, 22]]
    with make_engine(cfg, sd, f32) as e:
        solo = [replay(e, s, p) for s, p in zip(seqs, plans)]
        ids = [e.seq_open() for _ in seqs]
        at, got = [0] * 4, [[] for _ in seqs]
        plans = [list(p) for p in plans]
        step = 0
        while any(at[i] < len(seqs[i]) for i in range(4)):
            entries, who = [], []
            for i in range(4):
                if at[i] >= len(seqs[i]) or (step + i) % 5 == 4:  # every request sits out some steps
                    continue
                n = min(plans[i].pop(0) if plans[i] else 1, len(seqs[i]) - at[i])
                entries.append((ids[i], seqs[i][at[i]:at[i] + n], list(range(n))))
                who.append((i, n))
                at[i] += n
            step += 1
            if not entries:
                continue
            out, r = e.seq_step(entries), 0
            for i, n in who:
                got[i].append(out[r:r + n])
                r += n
        for sid in ids:
            e.seq_close(sid)
    for i in range(4):
        g = np.concatenate(got[i])
        assert row_err(g, want[i]).max() < TOL[f32]
        assert row_err(g, solo[i]).max() < (1e-5 if f32 else 3e-2)


def test_many_short_portions_in_one_step():
    # more tokens of short entries than one block of the per-head products takes, between entries that are expanded
    cfg = ref.random_config()
    sd = ref.random_state_dict(cfg, seed=35)
    o = ref.KamivikOracle(cfg, sd)
    lens = (40, 63, 2, 90, 50, 1, 63, 70, 30)
    seqs = [tokens(120 + i, n + 20, cfg["vocab"]) for i, n in enumerate(lens)]
    with make_engine(cfg, sd, 0, max_seqs=len(lens), ctx=512) as e:
        ids = [e.seq_open() for _ in lens]
        for sid, s in zip(ids, seqs):
            e.seq_step([(sid, s[:20], [])])
        out = e.seq_step([(sid, s[20:], list(range(len(s) - 20))) for sid, s in zip(ids, seqs)])
        r = 0
        for s in seqs:
            n = len(s) - 20
            assert row_err(out[r:r + n], o.forward(s)[20:]).max() < TOL[0]
            r += n


@pytest.mark.parametrize("f32", [1, 0])
def test_pages_and_slots_are_reused(f32):
    cfg = ref.random_config(order=((FULL, True), (WIN, False), (FULL, False)))
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=37), [0, 1])
    o = ref.KamivikOracle(cfg, sd)
    with make_engine(cfg, sd, f32, max_seqs=2, ctx=192, pool=256) as e:  # 4 pages, 2 sequences
        total = e.stats()["kv_pages_total"]
        assert total == 4
        for rnd in range(4):  # every pass reuses the pages and slots the previous one gave back
            a, b = tokens(40 + rnd, 130, cfg["vocab"]), tokens(50 + rnd, 60, cfg["vocab"])
            if rnd % 2 == 0:  # a row left behind by the last owner of a page would stand out
                a[::7] = [cfg["vocab"] - 1] * len(a[::7])
            sa, sb = e.seq_open(), e.seq_open()
            with pytest.raises(hb.HBError):
                e.seq_open()
            g1 = e.seq_step([(sa, a[:100], list(range(100))), (sb, b[:33], list(range(33)))])
            g2 = e.seq_step([(sa, a[100:], list(range(30))), (sb, b[33:], list(range(27)))])
            assert e.stats()["kv_pages_free"] == 0  # 3 + 1 pages
            e.seq_close(sa)
            e.seq_close(sb)
            assert e.stats()["kv_pages_free"] == total
            assert row_err(np.concatenate([g1[:100], g2[:30]]), o.forward(a)).max() < TOL[f32]
            assert row_err(np.concatenate([g1[100:], g2[30:]]), o.forward(b)).max() < TOL[f32]


@pytest.mark.parametrize("f32", [1, 0])
def test_greedy_generation_through_the_scheduler(f32):
    cfg = ref.random_config(vocab=200, order=((FULL, True), (WIN, True), (WIN, False), (FULL, True)))
    sd = ref.random_state_dict(cfg, seed=41)
    o = ref.KamivikOracle(cfg, sd)
    prompts = [tokens(60 + i, n, cfg["vocab"]) for i, n in enumerate((70, 5, 129))]
    with make_engine(cfg, sd, f32, max_seqs=4, ctx=256) as e:
        rids, outs = e.generate(prompts, hb.Sampling(max_tokens=24, capture=CAPTURE_STEP_LOGITS | CAPTURE_PROMPT_LOGITS))
        for p, rid, out in zip(prompts, rids, outs):
            rows = e.captured_logits(rid, CAPTURE_STEP_LOGITS)
            assert row_err(e.captured_logits(rid, CAPTURE_PROMPT_LOGITS), o.forward(p)).max() < TOL[f32]
            # teacher-forced comparison of every step's logits; ids must agree wherever the oracle's margin is clear
            st = o.new_state()
            z = o.forward(p, st)[-1]
            for k, t in enumerate(out):
                assert row_err(rows[k][None], z[None]).max() < TOL[f32]
                top2 = np.sort(z)[-2:]
                if top2[1] - top2[0] > 4 * TOL[f32] * np.sqrt((z * z).mean()):
                    assert t == int(np.argmax(z)), (k, t)
                z = o.forward([t], st)[-1]
        assert e.stats()["kv_pages_free"] == e.stats()["kv_pages_total"]


def test_continuous_batching_and_mixed_steps_match_solo_runs():
    cfg = ref.random_config(vocab=200)
    sd = ref.random_state_dict(cfg, seed=43)
    prompts = [tokens(80 + i, n, cfg["vocab"]) for i, n in enumerate((90, 17, 40, 66, 3, 120))]
    sp = hb.Sampling(max_tokens=12)
    with make_engine(cfg, sd, 1, max_seqs=4, ctx=256) as e:
        solo = [e.generate([p], sp)[1][0] for p in prompts]
        _, together = e.generate(prompts, sp)  # more prompts than slots: admission waits for finished sequences
        assert together == solo
    with make_engine(cfg, sd, 1, max_seqs=4, ctx=256, batched=128, decode_with_prefill=1, mixed_step_tokens=64) as e:
        _, mixed = e.generate(prompts, sp)  # prompts cut into 64-token portions beside the running sequences' tokens
        assert e.stats()["steps_mixed"] > 0
        assert mixed == solo
    with make_engine(cfg, sd, 1, max_seqs=4, ctx=256, use_cuda_graphs=1) as e:
        _, graphed = e.generate(prompts, sp)  # decode steps replayed from CUDA graphs (one per batch size)
        assert e.stats()["graph_launches"] > 0
        assert graphed == solo
    with make_engine(cfg, sd, 0, max_seqs=4, ctx=256, use_cuda_graphs=1) as e:  # serving mode: replayed steps, step by step
        o = ref.KamivikOracle(cfg, sd)
        rids, outs = e.generate(prompts[:3], hb.Sampling(max_tokens=40, capture=CAPTURE_STEP_LOGITS))
        for p, rid, out in zip(prompts, rids, outs):
            want = o.forward(p + out)[len(p) - 1:len(p) - 1 + len(out)]
            assert row_err(e.captured_logits(rid, CAPTURE_STEP_LOGITS), want).max() < TOL[0]


def test_unused_gain_is_skipped_and_bad_descriptions_are_rejected():
    cfg = ref.random_config()  # the last layer has no feed-forward
    sd = ref.random_state_dict(cfg, seed=71)
    toks = tokens(13, 40, cfg["vocab"])
    want = ref.KamivikOracle(cfg, sd).forward(toks)
    sd["l2.ls2"] = np.full(cfg["width"], 3.0, np.float32)
    with make_engine(cfg, sd, 1) as e:
        assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[1]
    desc = weights_io.desc_from_hf_config(cfg)
    with hb.Engine(hb.EngineConfig(device=0, max_seqs=2, max_ctx=128, max_batched_tokens=128)) as e:
        e.load_random(desc, seed=5)
        _, outs = e.generate([tokens(1, 20, cfg["vocab"])], hb.Sampling(max_tokens=4))
        assert len(outs[0]) == 4
    for edit in (lambda d: setattr(d.layers[1], "window", 0), lambda d: setattr(d.layers[0], "rope_dims", 10), lambda d: setattr(d.layers[0], "mask", 1),
                 lambda d: setattr(d.layers[0], "shared_ff", 8), lambda d: setattr(d, "norm_place", 1), lambda d: setattr(d.layers[0], "top_k", 7)):
        bad = weights_io.desc_from_hf_config(cfg)
        edit(bad)
        with hb.Engine(hb.EngineConfig(device=0, max_seqs=2, max_ctx=128, max_batched_tokens=128)) as e:
            with pytest.raises(hb.HBError):
                e.load_random(bad, seed=5)


def test_runtime_serves_a_checkpoint_folder(tmp_path):
    from helix_b200.runtime import B200Runtime, B200RuntimeParams
    cfg = ref.random_config(vocab=200)
    sd = ref.random_state_dict(cfg, seed=53)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    weights_io.write_safetensors(tmp_path / "model.safetensors", sd)
    rt = B200Runtime(B200RuntimeParams(model=str(tmp_path), context_length=256, serve_http=False,
                                       args=["--max-num-seqs", "4", "--max-num-batched-tokens", "256"]))
    rt.start()
    try:
        e = rt.engine
        prompt = tokens(9, 50, cfg["vocab"])
        rid = e.submit(prompt, hb.Sampling(max_tokens=8, capture=CAPTURE_STEP_LOGITS))
        out, fin = [], 0
        while not fin:
            assert e.wait(rid, 20000)
            t, fin = e.poll(rid)
            out += t
        rows = e.captured_logits(rid, CAPTURE_STEP_LOGITS)
        want = ref.KamivikOracle(cfg, sd).forward(prompt + out)[len(prompt) - 1:len(prompt) - 1 + len(out)]
        assert len(out) == 8 and row_err(rows, want).max() < TOL[0]  # teacher-forced on the engine's own ids (serving mode)
    finally:
        rt.stop()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_command(tmp_path, dtype):
    # bin/trace_run over a checkpoint folder: portions beside single tokens, requests that end and whose pages and slot the
    # next request takes, steps without wanted rows; the pool holds exactly what the live requests need (64-token pages)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = ref.random_config(vocab=120, order=((WIN, True), (FULL, True), (FULL, False), (WIN, True)))
    sd = ref.random_state_dict(cfg, seed=61)
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    weights_io.write_safetensors(model / "model.safetensors", sd)
    o = ref.KamivikOracle(cfg, sd)
    seqs = {k: tokens(90 + i, n, cfg["vocab"]) for i, (k, n) in enumerate((("a", 75), ("b", 40), ("c", 66), ("d", 9), ("e", 30)))}
    want = {k: o.forward(v) for k, v in seqs.items()}
    steps = [
        dict(step=0, entries=[dict(id="a", tokens=seqs["a"][:70], want=[0, 63, 64, 69])], end=[]),
        dict(step=1, entries=[dict(id="a", tokens=seqs["a"][70:71], want=[0]), dict(id="b", tokens=seqs["b"][:38], want=[])], end=[]),
        dict(step=2, entries=[dict(id="b", tokens=seqs["b"][38:], want=[1]), dict(id="a", tokens=seqs["a"][71:73], want=[0, 1]),
                              dict(id="c", tokens=seqs["c"][:2], want=[1]), dict(id="d", tokens=seqs["d"], want=[8])], end=["b", "d"]),
        dict(step=3, entries=[dict(id="c", tokens=seqs["c"][2:], want=[0, 61, 63]), dict(id="a", tokens=seqs["a"][73:], want=[1]),
                              dict(id="e", tokens=seqs["e"][:29], want=[28])], end=["a"]),
        dict(step=4, entries=[dict(id="e", tokens=seqs["e"][29:], want=[0])], end=["c", "e"]),
    ]
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "320"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(5)]
    at = {k: 0 for k in seqs}
    for s in steps:
        rows = []
        for en in s["entries"]:
            rows += [want[en["id"]][at[en["id"]] + w] for w in en["want"]]
            at[en["id"]] += len(en["tokens"])
        got = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(len(rows), cfg["vocab"])
        assert row_err(got, np.stack(rows)).max() < TOL[1 if dtype == "float32" else 0], s["step"]
