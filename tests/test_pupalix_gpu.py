"""Pupalix layer-list decoders through the engine (driven sequences and the scheduler) against the float64 oracle.

Every test builds its own small configuration and random bf16-representable weights (oracle/pupalix_ref.py; router choices are
made clear there, so no comparison rests on a close call); the engine runs them in its exact mode (fp32 weights, cache and
products), where a key left out, a block off by one, a state of the wrong pass or a wrong mix must show, and in its serving mode
(bf16 weights / cache rows / GEMM operands; fused attention kernels where the shapes fit them, the per-token kernels elsewhere)
with a rounding-sized bound.
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
from oracle import pupalix_ref as ref
from oracle.pupalix_ref import GQA, LATENT, LIGHT, dense_cfg, gqa_cfg, latent_cfg, light_cfg, moe_cfg

pytestmark = pytest.mark.gpu

TOL = {1: 2e-4, 0: 6e-2}  # compute_f32 -> bound on rms(diff) / rms(expected) per logits row


def row_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean(-1))


def make_engine(cfg, sd, f32, max_seqs=4, ctx=512, pool=0, batched=0, **kw):
    desc = weights_io.desc_from_hf_config(copy.deepcopy(cfg), {k: v.shape for k, v in sd.items()}, compute_f32=bool(f32))
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


def alone(kind, ff=None, **kw):
    return dict(dict(order=((kind, ff),), loop=None), **kw)


CONFIGS = {
    "default": dict(),
    "lightning_alone": alone(LIGHT),
    "latent_alone": alone(LATENT),
    "attention_alone": alone(GQA),
    "dense_alone": alone(LIGHT, "dense"),
    "experts_on_attention": alone(GQA, "moe"),
    "experts_on_latent": alone(LATENT, "moe"),
    # copies of the stream: one, two, four (in registers), five and sixteen (any number); a single plain stream is below
    "one_copy": dict(streams=1),
    "two_copies": dict(streams=2),
    "four_copies": dict(streams=4, loop=None),
    "five_copies": dict(streams=5, loop=(0, 2, 2)),
    "sixteen_copies": dict(streams=16, loop=None, order=((LIGHT, "dense"), (GQA, "moe"))),
    # loops: everything, one layer, the end, three passes, one pass
    "loop_over_everything": dict(loop=(0, 4, 2)),
    "loop_over_one_layer": dict(loop=(0, 1, 4)),
    "loop_at_the_end": dict(loop=(2, 4, 3)),
    "one_pass": dict(loop=(1, 3, 1)),
    # nothing a multiple of 8: every product takes the CUDA-core GEMM, attention the per-token kernels
    "odd_sizes": dict(width=91, vocab=131, ff=50, latent=latent_cfg(heads=5, dim=9, rot_dim=6, vdim=7, kv_rank=22), gqa=gqa_cfg(heads=6, kv_heads=2, dim=13),
                      light=light_cfg(heads=3, dim=7, vdim=11), moe=moe_cfg(5, 2, 21, None), buckets=13),
    # values a model may make equal or one
    "equal_sizes": dict(latent=latent_cfg(heads=2, dim=32, rot_dim=32, vdim=32, kv_rank=32), gqa=gqa_cfg(heads=2, kv_heads=2, dim=32),
                        light=light_cfg(heads=2, dim=32, vdim=32), width=128, ff=128, moe=moe_cfg(4, 2, 128, (2, 1)), buckets=120),
    "neutral_constants": dict(streams=1, embed_scale=1.0, logit_scale=1.0, logit_cap=None, moe=moe_cfg(1, 1, 40, (1, 1)), mul=(0, 1), buckets=1,
                              latent=latent_cfg(scale=1.0, scaling=(1.0, 60, 8.0, 1.0)), gqa=gqa_cfg(scale=1.0, softcap=None), loop=(0, 4, 1)),
    "no_options": dict(latent=latent_cfg(scaling=None), gqa=gqa_cfg(block=None, softcap=None), moe=moe_cfg(groups=None), logit_cap=None, loop=None),
    "one_head": dict(latent=latent_cfg(heads=1, dim=64, rot_dim=16, vdim=72, kv_rank=64), gqa=gqa_cfg(heads=1, kv_heads=1, dim=40), light=light_cfg(heads=1, dim=64, vdim=16)),
    "many_heads": dict(latent=latent_cfg(heads=17, dim=8, rot_dim=8, vdim=8, kv_rank=32), gqa=gqa_cfg(heads=14, kv_heads=2, dim=8), light=light_cfg(heads=19, dim=8, vdim=16)),
    "single_key_head": dict(gqa=gqa_cfg(heads=8, kv_heads=1, dim=64)),
    "decays_at_the_ends": alone(LIGHT, "dense", light=light_cfg(heads=4, decay=(0.0, 1.0, 0.5, 0.9999))),
    "wide_linear_heads": alone(LIGHT, "dense", width=128, light=light_cfg(heads=2, dim=200, vdim=136)),
    "narrow_linear_heads": alone(LIGHT, "dense", light=light_cfg(heads=5, dim=4, vdim=20)),
    # one head of 128 x 128 and of 64 x 64 keys and values: the fused attention kernels, blocks and caps as parameters
    "fused_128": dict(width=128, gqa=gqa_cfg(heads=4, kv_heads=2, dim=128, block=50), latent=latent_cfg(heads=3, dim=128, rot_dim=64, vdim=128, kv_rank=512), ff=128,
                      light=light_cfg(heads=2, dim=128, vdim=128)),
    "fused_64": dict(width=128, gqa=gqa_cfg(heads=6, kv_heads=6, dim=64, block=77, softcap=8.0), latent=latent_cfg(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128),
                     light=light_cfg(heads=3, dim=64, vdim=64), ff=64, moe=moe_cfg(8, 3, 64, (4, 3))),
    "block_of_one": dict(gqa=gqa_cfg(block=1)),
    "block_of_two": dict(gqa=gqa_cfg(block=2)),
    "block_of_a_page": dict(gqa=gqa_cfg(block=64)),
    "block_beyond_the_prompt": dict(gqa=gqa_cfg(block=400)),
    "every_expert_chosen": dict(moe=moe_cfg(4, 4, 40, (2, 2))),
    "one_expert_of_one_group": dict(moe=moe_cfg(9, 1, 40, (3, 1))),
    "groups_of_one": dict(moe=moe_cfg(8, 3, 40, (8, 5))),
    "many_experts": dict(moe=moe_cfg(72, 6, 24, (9, 4)), width=160),  # router wider than one MMA tile
    "ten_of_twenty": dict(moe=moe_cfg(20, 10, 40, (4, 3)), width=128),  # more expert rows per token than the residual step keeps in registers
    "layers_differ": dict(order=((GQA, "moe"), (LIGHT, None), (LATENT, "dense"), (GQA, None), (LIGHT, "moe")), loop=(1, 4, 2),
                          per_layer={2: latent_cfg(heads=2, dim=40, rot_dim=24, vdim=56, kv_rank=104, base=50.0, scaling=(8.0, 30, 4.0, 0.5), scale=0.3),
                                     3: gqa_cfg(heads=6, kv_heads=3, dim=16, block=90, softcap=5.0), 4: light_cfg(heads=2, dim=16, vdim=48, decay=(0.99, 0.3))},
                          per_mlp={2: dense_cfg(200), 4: moe_cfg(4, 3, 64, None)}),
}


@pytest.mark.parametrize("f32", [1, 0])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_portions_match_oracle(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=3)
    toks = tokens(1, 150, cfg["vocab"])  # crosses two page borders
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, f32) as e:
        assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[f32]
        assert row_err(replay(e, toks, [97, 2, 50]), want).max() < TOL[f32]


@pytest.mark.parametrize("name", ["default", "layers_differ", "fused_128", "fused_64", "many_experts", "ten_of_twenty", "five_copies"])
def test_steps_of_hundreds_of_tokens(name):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=5)
    toks = tokens(2, 430, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[f32]
            assert row_err(replay(e, toks, [300, 2, 97, 2]), want).max() < TOL[f32]


@pytest.mark.parametrize("name,f32", [("default", 1), ("default", 0), ("fused_128", 0), ("fused_64", 0), ("odd_sizes", 0)])
def test_prefill_portions_and_single_tokens_agree(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=7)
    toks = tokens(3, 140, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, f32) as e:
        whole = replay(e, toks, [len(toks)])
        for cuts in ([64, 64], [63, 2, 2, 61], [19, 20, 21, 2, 45], [1, 1, 1, 2, 3, 64, 5], [2, 2, 2, 3, 2], []):
            got = replay(e, toks, cuts)
            assert row_err(got, want).max() < TOL[f32], cuts
            assert row_err(got, whole).max() < (1e-5 if f32 else 4e-2), cuts  # the same positions, cut differently: rounding only


def with_block(cfg, size):
    c = copy.deepcopy(cfg)
    c["layers"][0]["mixer"]["mask"] = dict(size=size)
    return c


@pytest.mark.parametrize("dim", [24, 64, 128])
@pytest.mark.parametrize("block,at", [(64, 0), (64, 70), (50, 99), (37, 74), (100, 130), (2, 62), (130, 5)])
def test_block_edges_in_prompts_and_in_decoding(block, at, dim):
    # a marker token every head looks at while it is in the same block: the block's last position sees it, the next one does not
    cfg = ref.random_config(**alone(GQA, gqa=gqa_cfg(block=block, dim=dim, scale=0.5), width=128))
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=11), [0])
    edge = (at // block + 1) * block
    toks = tokens(4, edge + 40, cfg["vocab"])
    toks[at] = cfg["vocab"] - 1
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    plain = list(toks)
    plain[at] = 3
    assert row_err(ref.PupalixOracle(cfg, sd).forward(plain)[edge - 1], want[edge - 1]) > 3 * TOL[0]  # seen just inside ...
    if edge > at + 2:  # (the pair row of the token behind the marker differs as well)
        assert row_err(ref.PupalixOracle(cfg, sd).forward(plain)[edge], want[edge]) < 1e-9             # ... and not just outside
        assert row_err(ref.PupalixOracle(with_block(cfg, edge + 1), sd).forward(toks)[edge], want[edge]) > 3 * TOL[0]
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            # one prompt; decoding over the edge; portions that start or end on it; portions of two
            for cuts in ([len(toks)], [max(1, edge - 3)], [edge - 1, 2, 2, 2], [edge, 64], [2] * (len(toks) // 2 + 1), [max(1, edge - 66), 66, 2]):
                assert row_err(replay(e, toks, cuts), want).max() < TOL[f32], cuts


@pytest.mark.parametrize("name", ["default", "fused_128", "odd_sizes"])
def test_far_keys_and_page_borders(name):
    # markers at the first token, at page borders and in between; the latent layer's queries hundreds of positions on still see them
    cfg = ref.random_config(**dict(CONFIGS[name], order=((LATENT, "moe"), (LATENT, None)), loop=None))
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=13), [0])
    for at in (0, 63, 64, 150):
        toks = tokens(5, 400, cfg["vocab"])
        o = ref.PupalixOracle(cfg, sd)
        plain = o.forward(toks)
        toks[at] = cfg["vocab"] - 1
        want = o.forward(toks)
        assert row_err(plain[-100:], want[-100:]).min() > 2 * TOL[0]  # what losing the far key would look like
        for f32 in (1, 0):
            with make_engine(cfg, sd, f32) as e:
                for cuts in ([len(toks)], [255, 2, 1, 1, 1, 2, 64], [64, 64, 128, 130]):
                    assert row_err(replay(e, toks, cuts), want).max() < TOL[f32], cuts


@pytest.mark.parametrize("light", [light_cfg(), light_cfg(heads=2, dim=128, vdim=128, decay=(0.999, 0.97)), light_cfg(heads=3, dim=64, vdim=72, decay=(1.0, 0.6, 0.0))])
def test_recurrent_state_across_portions_of_every_size(light):
    # decays near one keep early tokens in the state for hundreds of positions; portions end inside, on and behind chunk borders
    cfg = ref.random_config(**alone(LIGHT, "dense", light=light, width=128))
    sd = ref.random_state_dict(cfg, seed=19)
    toks = tokens(7, 420, cfg["vocab"])
    o = ref.PupalixOracle(cfg, sd)
    want = o.forward(toks)
    other = list(toks)
    other[3] = (toks[3] + 7) % (cfg["vocab"] - 1)
    assert row_err(o.forward(other)[-1], want[-1]) > 5 * TOL[1]  # four hundred positions on
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            for cuts in ([420], [1, 63, 64, 65, 127, 100], [128, 128, 128, 36], [16, 17, 15, 32, 33, 31, 276], [2, 3, 200, 2, 2, 150], [64] * 6):
                assert row_err(replay(e, toks, cuts), want).max() < (TOL[1] if f32 else 3e-2), cuts


def test_rotation_at_large_positions_and_its_scaling():
    # short wavelengths: positions in the hundreds turn many times, on the key part that all heads share and on the queries
    lat = lambda **kw: latent_cfg(base=30.0, scale=0.3, rot_dim=16, **kw)
    cfg = ref.random_config(**alone(LATENT, latent=lat(scaling=(3.0, 200, 20.0, 2.0))))
    sd = ref.random_state_dict(cfg, seed=23)
    toks = tokens(8, 400, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    for sc in (None, (3.0, 200, 20.0, 1.0), (3.0, 200, 40.0, 2.0), (3.0, 300, 20.0, 2.0), (2.5, 200, 20.0, 2.0)):
        c = ref.random_config(**alone(LATENT, latent=lat(scaling=sc)))
        assert row_err(ref.PupalixOracle(c, sd).forward(toks)[5:], want[5:]).max() > 20 * TOL[1], sc
    for f32, cuts in ((1, [len(toks)]), (1, [390]), (0, [199, 2]), (0, [len(toks)])):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, cuts), want).max() < TOL[f32]


def test_first_tokens_of_a_sequence():
    # position 0 takes the last bigram row, sees itself alone, and starts from a zero state
    cfg = ref.random_config()
    sd = ref.random_state_dict(cfg, seed=25)
    toks = tokens(9, 12, cfg["vocab"])
    o = ref.PupalixOracle(cfg, sd)
    want = o.forward(toks)
    other = dict(sd, bigram=sd["bigram"].copy())
    other["bigram"][-1] = other["bigram"][0]
    assert row_err(ref.PupalixOracle(cfg, other).forward(toks)[0], want[0]) > 3 * TOL[0]
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32, max_seqs=1) as e:
            for cuts in ([], [1, 2, 2], [2, 3], [len(toks)]):
                assert row_err(replay(e, toks, cuts), want).max() < TOL[f32]


def test_alternative_readings_differ_and_the_engine_follows_the_oracle():
    cfg = ref.random_config()
    sd = ref.random_state_dict(cfg, seed=27)
    toks = tokens(10, 60, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)

    def alt(edit_cfg=None, edit_sd=None):
        c, s = copy.deepcopy(cfg), {k: v.copy() for k, v in sd.items()}
        if edit_cfg:
            edit_cfg(c)
        if edit_sd:
            edit_sd(s)
        return ref.PupalixOracle(c, s).forward(toks)

    def each(s, end, f):
        for k in [k for k in s if k.endswith(end)]:
            s[k] = f(s[k])

    swap = lambda c: c["embedding"]["bigram"].update(mul_prev=5, mul_cur=31)
    for other in (alt(swap), alt(lambda c: c["embedding"].update(scale=2.4)), alt(lambda c: c.update(logit_scale=0.6)), alt(lambda c: c.update(logit_softcap=14.0)),
                  alt(lambda c: c["layers"][2]["mixer"].update(softcap=3.0)), alt(lambda c: c["loop"].update(times=3)), alt(lambda c: c.pop("loop")),
                  alt(lambda c: c["layers"][0]["mixer"].update(decay=[0.93, 0.5, 0.998])), alt(lambda c: c["layers"][1]["mlp"]["router"].pop("groups")),
                  alt(None, lambda s: each(s, ".mix.k.norm", np.ones_like)), alt(None, lambda s: each(s, "hc1.mix", np.transpose)),
                  alt(None, lambda s: each(s, "hc2.in", np.ones_like)), alt(None, lambda s: each(s, "hc2.out", np.ones_like))):
        assert row_err(other, want).max() > 20 * TOL[1]
    act = ref.gelu_tanh
    import math
    erf = np.vectorize(math.erf, otypes=[float])
    ref.gelu_tanh = lambda z: 0.5 * z * (1 + erf(z / math.sqrt(2)))
    try:
        assert row_err(ref.PupalixOracle(cfg, sd).forward(toks), want).max() > 1e-4  # the erf form is another function
    finally:
        ref.gelu_tanh = act
    for f32 in (1, 0):
        with make_engine(cfg, sd, f32) as e:
            assert row_err(replay(e, toks, [33, 2]), want).max() < (5e-5 if f32 else TOL[0])


def test_one_plain_stream():
    # no copies: x <- x + mixer(norm1 x), x <- x + ff(norm2 x); the same as one copy whose weights are all one
    cfg = ref.random_config(streams=1)
    sd = ref.random_state_dict(cfg, seed=29)
    for k in sd:
        if ".hc" in k:
            sd[k] = np.ones_like(sd[k])
    toks = tokens(11, 90, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    bare = {k: v for k, v in sd.items() if ".hc" not in k}
    for f32 in (1, 0):
        with make_engine(cfg, bare, f32) as e:
            assert row_err(replay(e, toks, [61, 2]), want).max() < TOL[f32]


def test_long_decoding_over_pages():
    cfg = ref.random_config()
    sd = ref.random_state_dict(cfg, seed=31)
    toks = tokens(8, 230, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    with make_engine(cfg, sd, 1) as e:
        assert row_err(replay(e, toks, [10]), want).max() < TOL[1]  # 220 single-token steps
    with make_engine(cfg, sd, 0, use_cuda_graphs=1) as e:
        assert row_err(replay(e, toks, [10]), want).max() < TOL[0]


@pytest.mark.parametrize("name,f32", [("default", 1), ("default", 0), ("fused_128", 0), ("fused_64", 0), ("odd_sizes", 1), ("odd_sizes", 0)])
def test_mixed_batches_match_each_request_alone(name, f32):
    cfg = ref.random_config(**CONFIGS[name])
    sd = ref.random_state_dict(cfg, seed=33)
    o = ref.PupalixOracle(cfg, sd)
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
        assert row_err(g, solo[i]).max() < (1e-5 if f32 else 4e-2)


@pytest.mark.parametrize("f32", [1, 0])
def test_pages_and_slots_are_reused(f32):
    cfg = ref.random_config(order=((LATENT, "moe"), (GQA, None), (LIGHT, "dense")), gqa=gqa_cfg(scale=0.5), loop=(0, 2, 2))
    sd = ref.plant_marker(cfg, ref.random_state_dict(cfg, seed=37), [0, 1])
    o = ref.PupalixOracle(cfg, sd)
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
    cfg = ref.random_config(vocab=200)
    sd = ref.random_state_dict(cfg, seed=41)
    o = ref.PupalixOracle(cfg, sd)
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
    with make_engine(cfg, sd, 1, max_seqs=4, ctx=256, pool=320) as e:  # a small pool: sequences are preempted and recomputed
        _, tight = e.generate(prompts, sp)
        assert tight == solo
    with make_engine(cfg, sd, 0, max_seqs=4, ctx=256, use_cuda_graphs=1) as e:  # serving mode: replayed steps, step by step
        o = ref.PupalixOracle(cfg, sd)
        rids, outs = e.generate(prompts[:3], hb.Sampling(max_tokens=40, capture=CAPTURE_STEP_LOGITS))
        for p, rid, out in zip(prompts, rids, outs):
            want = o.forward(p + out)[len(p) - 1:len(p) - 1 + len(out)]
            assert row_err(e.captured_logits(rid, CAPTURE_STEP_LOGITS), want).max() < TOL[0]


def test_unused_tensors_are_skipped_and_bad_descriptions_are_rejected():
    cfg = ref.random_config(per_mlp={3: None})
    sd = ref.random_state_dict(cfg, seed=71)
    toks = tokens(13, 40, cfg["vocab"])
    want = ref.PupalixOracle(cfg, sd).forward(toks)
    sd["l3.norm2"] = np.full(cfg["width"], 3.0, np.float32)
    sd["l3.hc2.mix"] = np.full((3, 3), 3.0, np.float32)
    with make_engine(cfg, sd, 1) as e:
        assert row_err(replay(e, toks, [len(toks)]), want).max() < TOL[1]
    desc = weights_io.desc_from_hf_config(cfg)
    with hb.Engine(hb.EngineConfig(device=0, max_seqs=2, max_ctx=128, max_batched_tokens=128)) as e:
        e.load_random(desc, seed=5)
        _, outs = e.generate([tokens(1, 20, cfg["vocab"])], hb.Sampling(max_tokens=4))
        assert len(outs[0]) == 4

    def layer(i, **kw):
        return lambda d: [setattr(d.layers[i], k, v) for k, v in kw.items()]

    for edit in (layer(0, head_decay=()), layer(0, head_decay=(0.5, 1.5, 0.5)), layer(0, dim=300), layer(1, rope_original=0), layer(1, route_groups=4),
                 layer(1, route_keep=0), layer(1, attn_flags=4096 | 2048 | 8), layer(2, window=0), lambda d: setattr(d, "streams", 17),
                 lambda d: setattr(d, "loop_stop", 5), lambda d: setattr(d, "loop_start", 3), lambda d: setattr(d, "bigram_mul_prev", -1),
                 lambda d: setattr(d, "norm_place", 1), lambda d: setattr(d, "plain_gains", 0)):
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
        want = ref.PupalixOracle(cfg, sd).forward(prompt + out)[len(prompt) - 1:len(prompt) - 1 + len(out)]
        assert len(out) == 8 and row_err(rows, want).max() < TOL[0]  # teacher-forced on the engine's own ids (serving mode)
    finally:
        rt.stop()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_command(tmp_path, dtype):
    # bin/trace_run over a checkpoint folder: portions beside single tokens, requests that end and whose pages and slot the
    # next request takes, steps without wanted rows; the pool holds exactly what the live requests need (64-token pages)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = ref.random_config(vocab=120, order=((GQA, "moe"), (LATENT, "dense"), (LIGHT, None), (LATENT, "moe")), loop=(1, 3, 2))
    sd = ref.random_state_dict(cfg, seed=61)
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    weights_io.write_safetensors(model / "model.safetensors", sd)
    o = ref.PupalixOracle(cfg, sd)
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
