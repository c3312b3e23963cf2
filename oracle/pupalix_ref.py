"""Plain, slow float64 restatement of the Pupalix decoder (numpy only; one function per mechanism).

The design: a scaled embedding plus a row picked by the (previous token, token) pair; several copies of the residual stream
that every sublayer reads through one learned combination and writes back through another, mixing the copies as it does;
pre-norms; three mixers — attention over a cached low-rank latent with a YaRN-scaled rotation of the key part all heads share,
grouped-query attention inside blocks of positions whose values are its key projections, and linear attention with one constant
decay per head; tanh-GELU feed-forwards or group-limited mixtures of SiLU experts; a run of layers that is passed through
several times with the same weights, each pass with rows and state of its own; logits from the embedding table.  Notation: T
tokens, W width, S stream copies, H heads, G key heads, Dk / Dr / Dv unrotated / rotated / value sizes per head, R latent rank.
Nothing here is shared with the CUDA path; the GPU tests compare the engine against these functions.
"""
import math

import numpy as np

F = np.float64
LATENT, GQA, LIGHT = "latent_attention", "attention", "lightning"


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    x = np.asarray(x, F)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * np.asarray(w, F)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def cap(z, c):
    return c * np.tanh(z / c) if c else z


# ------------------------------------------------------------------ embedding, streams
def embed(tokens, prev, table, bigram, scale, mul_prev, mul_cur):
    """prev: the token before tokens[0] (None at the start of a sequence).  Rows 0 .. B-1 of `bigram` (B = rows - 1) belong to
    pairs, row B to a token without a predecessor."""
    B = bigram.shape[0] - 1
    before = [prev] + list(tokens[:-1])
    rows = [B if p is None else (int(p) * mul_prev + int(t) * mul_cur) % B for p, t in zip(before, tokens)]
    return table[np.asarray(tokens)] * scale + bigram[rows]


def read_streams(xs, w):
    """u = sum_s w_s x_s; xs [S, T, W]"""
    return np.einsum("s,stw->tw", w, xs)


def write_streams(xs, y, mix, out):
    """every copy from the old ones: x_t <- sum_s mix[s, t] x_s + out_t y"""
    return np.einsum("st,snw->tnw", mix, xs) + out[:, None, None] * y[None]


# ------------------------------------------------------------------ rotation
def yarn(dims, base, sc):
    """(frequencies [dims / 2], factor of cos and sin)"""
    i = np.arange(dims // 2, dtype=F)
    f = float(base) ** (-2.0 * i / dims)
    if not sc:
        return f, 1.0
    where = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(v, pos, rot):
    """Entries 2i and 2i + 1 of the last axis form a pair, i < dims / 2; the entries behind them stay."""
    v = np.array(v, F)
    dims = rot["dims"]
    f, mult = yarn(dims, rot["base"], rot.get("scaling"))
    a = np.asarray(pos, F)[..., None] * f
    c, s = np.cos(a) * mult, np.sin(a) * mult
    while c.ndim < v.ndim:  # head axes between the token axis and the last axis
        c, s = c[..., None, :], s[..., None, :]
    u, w = v[..., 0:dims:2].copy(), v[..., 1:dims:2].copy()
    v[..., 0:dims:2] = u * c - w * s
    v[..., 1:dims:2] = w * c + u * s
    return v


# ------------------------------------------------------------------ attention
def visible(pos, kpos, block):
    """[T, J] mask: earlier positions, of the same block of `block` positions (None: all of them)"""
    p, k = np.asarray(pos)[:, None], np.asarray(kpos)[None, :]
    return (k <= p) if block is None else (k <= p) & (k // block == p // block)


def softmax_seen(s, seen):
    """softmax over the last axis of s [T, H, J] restricted to seen [T, J]"""
    s = np.where(seen[:, None, :], s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def latent_row(h, p, m, pos):
    """What is kept per token: the normed latent [T, R] and the rotated shared key part [T, Dr]."""
    R = m["kv_rank"]
    d = h @ p["dkv"].T
    return rms_norm(d[:, :R], p["dkv.norm"], m["eps"]), rotate(d[:, R:], pos, m["rot"])


def latent_heads(h, p, m, pos, c, kr, kpos):
    """Head outputs [T, H, Dv]; c / kr / kpos: rows and positions of EVERY key so far (this call's tokens included)."""
    T = h.shape[0]
    H, Dk, Dr, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, Dk + Dr)
    qn, qr = q[:, :, :Dk], rotate(q[:, :, Dk:], pos, m["rot"])
    kn = (c @ p["uk"].T).reshape(-1, H, Dk)
    val = (c @ p["uv"].T).reshape(-1, H, Dv)
    s = (np.einsum("thd,jhd->thj", qn, kn) + np.einsum("thd,jd->thj", qr, kr)) * m["scale"]
    return np.einsum("thj,jhv->thv", softmax_seen(s, visible(pos, kpos, None)), val)


def gqa_rows(h, p, m):
    """keys (normed over the whole projection) and values (the projection as it is), [T, G, Dk]"""
    k = h @ p["k"].T
    shape = (h.shape[0], m["kv_heads"], m["dim"])
    return rms_norm(k, p["k.norm"], m["eps"]).reshape(shape), k.reshape(shape)


def gqa_heads(h, p, m, pos, k, v, kpos):
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms_norm(h @ p["q"].T, p["q.norm"], m["eps"]).reshape(T, H, D)
    own = np.arange(H) // (H // G)
    s = cap(np.einsum("thd,jhd->thj", q, k[:, own]) * m["scale"], m.get("softcap"))
    mask = m.get("mask")
    return np.einsum("thj,jhv->thv", softmax_seen(s, visible(pos, kpos, mask["size"] if mask else None)), v[:, own])


# ------------------------------------------------------------------ linear attention with constant decays
def lightning(h, p, m, state):
    """(concatenated heads [T, H * Dv] before norm and gate, state [H, Dk, Dv] behind the last token)"""
    T, H, Dk, Dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ p["q"].T).reshape(T, H, Dk), silu(h @ p["k"].T).reshape(T, H, Dk)
    v = silu(h @ p["v"].T).reshape(T, H, Dv)
    a = np.asarray(m["decay"], F)[:, None, None]
    out = np.empty((T, H, Dv), F)
    for t in range(T):
        state = a * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hd,hdv->hv", q[t], state)
    return out.reshape(T, -1), state


def lightning_readout(o, h, p, eps):
    return rms_norm(o, p["norm"], eps) * sigmoid(h @ p["g"].T)


# ------------------------------------------------------------------ feed-forwards
def dense(h, p):
    return (gelu_tanh(h @ p["gate"].T) * (h @ p["up"].T)) @ p["down"].T


def eligible(s, groups):
    """[T, E] mask of the experts of the best groups; a group's score is its largest"""
    n, keep = groups["count"], groups["keep"]
    g = s.reshape(s.shape[0], n, -1).max(-1)
    best = np.argsort(-g, axis=-1, kind="stable")[:, :keep]
    ok = np.zeros(g.shape, bool)
    np.put_along_axis(ok, best, True, -1)
    return np.repeat(ok, s.shape[1] // n, axis=-1)


def route(h, router, r):
    """chosen experts [T, top] (largest first) and their scores, softmax over ALL experts"""
    z = h @ router.T
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    pick = np.where(eligible(s, r["groups"]), s, -1.0) if r.get("groups") else s
    ids = np.argsort(-pick, axis=-1, kind="stable")[:, :r["top"]]
    return ids, np.take_along_axis(s, ids, -1)


def route_margin(h, router, r):
    """how far (in logits) the closest choice is from another outcome, per token: between the last chosen and the best left out of
    the eligible experts, and between the last kept and the best dropped group"""
    z = h @ router.T
    out = np.full(len(z), np.inf)
    g = r.get("groups")
    if g and g["keep"] < g["count"]:
        top = -np.sort(-z.reshape(len(z), g["count"], -1).max(-1), axis=-1)
        out = np.minimum(out, top[:, g["keep"] - 1] - top[:, g["keep"]])
        z = np.where(eligible(z, g), z, -np.inf)
    z = -np.sort(-z, axis=-1)
    if z.shape[1] > r["top"]:
        out = np.minimum(out, z[:, r["top"] - 1] - z[:, r["top"]])
    return out


def expert(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def mixture(h, p, mlp):
    r = mlp["router"]
    ids, w = route(h, p["router"], r)
    out = np.zeros((h.shape[0], p["e0.down"].shape[0]), F)
    for e in range(r["experts"]):
        t, k = np.nonzero(ids == e)
        if len(t):
            np.add.at(out, t, w[t, k][:, None] * expert(h[t], p[f"e{e}.gate"], p[f"e{e}.up"], p[f"e{e}.down"]))
    return out


# ------------------------------------------------------------------ the model
def runs(cfg):
    """layer indices in the order they are run"""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    body = list(range(lp["start"], lp["stop"]))
    return list(range(lp["start"])) + body * lp["times"] + list(range(lp["stop"], n))


class PupalixOracle:
    """cfg: the checkpoint's config dict; sd: {tensor name: ndarray}.  `forward` runs a portion of one sequence from the
    state an earlier call left, so prefill, portions and token-by-token decoding are the same function called differently."""

    def __init__(self, cfg, sd):
        self.cfg = cfg
        self.sd = {k: np.asarray(v, F) for k, v in sd.items()}
        self.eps = cfg["norm"]["eps"]
        self._subs = {}

    def sub(self, prefix):
        if prefix not in self._subs:
            n = len(prefix)
            self._subs[prefix] = {k[n:]: v for k, v in self.sd.items() if k.startswith(prefix)}
        return self._subs[prefix]

    def new_state(self):
        return {"pos": 0, "prev": None, "rows": {}}

    def mixer(self, run, i, h, st, pos):
        """run: which pass over which layer (rows and state belong to it); i: the layer whose weights it uses"""
        ly = self.cfg["layers"][i]
        m, p = dict(ly["mixer"], eps=self.eps), self.sub(f"l{i}.mix.")
        if ly["type"] == LIGHT:
            S = st["rows"].get(run, np.zeros((m["heads"], m["dim"], m["vdim"]), F))
            o, st["rows"][run] = lightning(h, p, m, S)
            return lightning_readout(o, h, p, self.eps) @ p["o"].T
        new = latent_row(h, p, m, pos) if ly["type"] == LATENT else gqa_rows(h, p, m)
        if run in st["rows"]:
            new = tuple(np.concatenate([a, b]) for a, b in zip(st["rows"][run], new))
        st["rows"][run] = new
        heads = latent_heads if ly["type"] == LATENT else gqa_heads
        return heads(h, p, m, pos, *new, np.arange(len(new[0]))).reshape(h.shape[0], -1) @ p["o"].T

    def forward(self, tokens, st=None, taps=None, margins=None):
        """tokens -> logits [T, vocab]; st is updated in place.  taps / margins (lists) receive the summed stream after every layer
        run / every router's margins."""
        cfg, sd = self.cfg, self.sd
        st = self.new_state() if st is None else st
        pos = np.arange(st["pos"], st["pos"] + len(tokens))
        b = cfg["embedding"]["bigram"]
        x = embed(tokens, st["prev"], sd["embed"], sd["bigram"], cfg["embedding"]["scale"], b["mul_prev"], b["mul_cur"])
        xs = np.repeat(x[None], cfg["streams"], axis=0)
        for run, i in enumerate(runs(cfg)):
            mlp = cfg["layers"][i].get("mlp")
            h = rms_norm(read_streams(xs, sd[f"l{i}.hc1.in"]), sd[f"l{i}.norm1"], self.eps)
            xs = write_streams(xs, self.mixer(run, i, h, st, pos), sd[f"l{i}.hc1.mix"], sd[f"l{i}.hc1.out"])
            if mlp is not None:
                h = rms_norm(read_streams(xs, sd[f"l{i}.hc2.in"]), sd[f"l{i}.norm2"], self.eps)
                p = self.sub(f"l{i}.mlp.")
                if mlp["kind"] == "moe" and margins is not None:
                    margins.append(route_margin(h, p["router"], mlp["router"]))
                y = mixture(h, p, mlp) if mlp["kind"] == "moe" else dense(h, p)
                xs = write_streams(xs, y, sd[f"l{i}.hc2.mix"], sd[f"l{i}.hc2.out"])
            if taps is not None:
                taps.append(xs.sum(0))
        st["pos"] += len(tokens)
        st["prev"] = int(tokens[-1])
        z = rms_norm(xs.sum(0), sd["final.norm"], self.eps) @ sd["embed"].T * cfg.get("logit_scale", 1.0)
        return cap(z, cfg.get("logit_softcap"))


# ------------------------------------------------------------------ random checkpoints for tests
def latent_cfg(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, base=1000.0, scaling=(4.0, 60, 8.0, 1.0), scale=None):
    """scaling: (factor, original, fast, slow) or None"""
    rot = dict(dims=rot_dim, base=float(base))
    if scaling:
        rot["scaling"] = dict(factor=float(scaling[0]), original=int(scaling[1]), fast=float(scaling[2]), slow=float(scaling[3]))
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, rot=rot, scale=float(scale if scale is not None else (dim + rot_dim) ** -0.5))


def gqa_cfg(heads=4, kv_heads=2, dim=24, block=37, softcap=20.0, scale=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=float(scale if scale is not None else 2.0 * dim ** -0.5))
    if softcap:
        m["softcap"] = float(softcap)
    if block:
        m["mask"] = dict(size=block)
    return m


def light_cfg(heads=3, dim=24, vdim=40, decay=(0.5, 0.93, 0.998)):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=[float(decay[h % len(decay)]) for h in range(heads)])


def moe_cfg(experts=6, top=3, ff=40, groups=(3, 2)):
    r = dict(experts=experts, top=top)
    if groups:
        r["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=r)


def dense_cfg(ff=72):
    return dict(kind="dense", ff=ff)


DEFAULT_ORDER = ((LIGHT, "dense"), (LATENT, "moe"), (GQA, "dense"), (LIGHT, "moe"))


def random_config(width=96, vocab=120, order=DEFAULT_ORDER, latent=None, gqa=None, light=None, moe=None, ff=72, streams=3, loop=(1, 3, 2), buckets=97,
                  mul=(31, 5), embed_scale=2.5, logit_scale=0.5, logit_cap=12.0, eps=1e-5, per_layer=None, per_mlp=None):
    """order: (type, "dense" | "moe" | None) per layer; per_layer / per_mlp {i: dict}: that layer's mixer / feed-forward."""
    layers = []
    for i, (kind, f) in enumerate(order):
        mixer = {LATENT: latent or latent_cfg(), GQA: gqa or gqa_cfg(), LIGHT: light or light_cfg()}[kind]
        mlp = dense_cfg(ff) if f == "dense" else (moe or moe_cfg()) if f == "moe" else None
        layers.append(dict(type=kind, mixer=(per_layer or {}).get(i, mixer), mlp=(per_mlp or {}).get(i, mlp)))
    cfg = dict(architecture="Pupalix", width=width, vocab=vocab, layers=layers, norm=dict(eps=eps), streams=streams, logit_scale=float(logit_scale),
               embedding=dict(scale=float(embed_scale), bigram=dict(buckets=buckets, mul_prev=mul[0], mul_cur=mul[1])))
    if logit_cap:
        cfg["logit_softcap"] = float(logit_cap)
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def reserved(cfg):
    """leading stream entries that no sublayer writes: one per expert, then two for planted features"""
    return max([ly["mlp"]["router"]["experts"] for ly in cfg["layers"] if ly["mlp"] and ly["mlp"]["kind"] == "moe"] + [0]) + 2


def random_state_dict(cfg, seed=0):
    """Router choices are made by the leading stream entries, which hold a shuffled grid of values per token and keep its order
    through every mix of the copies, so that no choice is a close call; everything else is random."""
    from .weights import _rng, _t, to_bf16_f32
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    s = lambda n: 1.0 / math.sqrt(n)
    n_res = reserved(cfg)
    E0 = n_res - 2
    step = min(0.5, 4.0 / max(E0, 1))
    table = _t(seed, "embed", (V, W), 0.4)
    g = _rng(seed, "grid")
    for v in range(V):
        table[v, :E0] = (g.permutation(E0) - (E0 - 1) / 2.0) * step
    table[:, E0:n_res] = 0.0
    big = _t(seed, "bigram", (cfg["embedding"]["bigram"]["buckets"] + 1, W), 0.6)
    big[:, :n_res] = 0.0
    sd = {"embed": to_bf16_f32(table), "bigram": to_bf16_f32(big), "final.norm": _t(seed, "fn", (W,), 0.1, 1.0)}
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}."
        H, Dk, Dv = m["heads"], m["dim"], m["vdim"]
        o_rows = _t(seed, p + "o", (W, H * Dv), 1.5 * s(H * Dv))
        o_rows[:n_res] = 0.0
        sd[p + "mix.o"] = o_rows
        for q in (1, 2):
            if q == 2 and not ly["mlp"]:
                continue
            sd[p + f"norm{q}"] = _t(seed, p + f"n{q}", (W,), 0.1, 1.0)
            sd[p + f"norm{q}"][:n_res] = 1.0
            sd[p + f"hc{q}.in"] = to_bf16_f32(np.abs(_t(seed, p + f"hi{q}", (S,), 0.3, 1.0 / S)) + 0.05)
            sd[p + f"hc{q}.out"] = _t(seed, p + f"ho{q}", (S,), 0.5, 0.7)
            sd[p + f"hc{q}.mix"] = to_bf16_f32(np.abs(_t(seed, p + f"hm{q}", (S, S), 0.15)) + 0.75 * np.eye(S))
        if ly["type"] == LATENT:
            Dr, R = m["rot_dim"], m["kv_rank"]
            sd[p + "mix.q"] = _t(seed, p + "q", (H * (Dk + Dr), W), 1.5 * s(W))
            sd[p + "mix.dkv"] = _t(seed, p + "dkv", (R + Dr, W), 1.5 * s(W))
            sd[p + "mix.dkv.norm"] = _t(seed, p + "dkvn", (R,), 0.1, 1.0)
            sd[p + "mix.uk"] = _t(seed, p + "uk", (H * Dk, R), 1.5 * s(R))
            sd[p + "mix.uv"] = _t(seed, p + "uv", (H * Dv, R), 1.5 * s(R))
        elif ly["type"] == GQA:
            G = m["kv_heads"]
            sd[p + "mix.q"] = _t(seed, p + "q", (H * Dk, W), 1.5 * s(W))
            sd[p + "mix.k"] = _t(seed, p + "k", (G * Dk, W), 1.5 * s(W))
            sd[p + "mix.q.norm"] = _t(seed, p + "qn", (H * Dk,), 0.2, 1.0)
            sd[p + "mix.k.norm"] = _t(seed, p + "kn", (G * Dk,), 0.2, 1.0)
        else:
            for n, rows in (("q", H * Dk), ("k", H * Dk), ("v", H * Dv), ("g", H * Dv)):
                sd[p + "mix." + n] = _t(seed, p + n, (rows, W), 1.5 * s(W))
            sd[p + "mix.norm"] = _t(seed, p + "ln", (H * Dv,), 0.2, 1.0)
        if not ly["mlp"]:
            continue
        if ly["mlp"]["kind"] == "dense":
            units, Fn = [""], ly["mlp"]["ff"]
        else:
            E, Fn = ly["mlp"]["router"]["experts"], ly["mlp"]["expert"]["ff"]
            units = [f"e{e}." for e in range(E)]
            router = _t(seed, p + "router", (E, W), 0.05 * s(W))
            router[:, :n_res] = 0.0
            for e in range(E):
                router[e, e] = 4.0 / step / cfg["embedding"]["scale"]
            sd[p + "mlp.router"] = to_bf16_f32(router)
        for u in units:
            sd[p + f"mlp.{u}gate"] = _t(seed, p + f"{u}g", (Fn, W), 1.5 * s(W))
            sd[p + f"mlp.{u}up"] = _t(seed, p + f"{u}u", (Fn, W), 1.5 * s(W))
            down = _t(seed, p + f"{u}d", (W, Fn), (2.0 if u else 1.0) * s(Fn))
            down[:n_res] = 0.0
            sd[p + f"mlp.{u}down"] = down
    return sd


def plant_marker(cfg, sd, layers, strength=14.0):
    """Token vocab - 1 becomes a marker: in the named attention layers every head's score for it stands out wherever it is seen, and
    its value is unlike any other token's, so whether a position sees it shows in the logits."""
    from .weights import to_bf16_f32
    sd = {k: v.copy() for k, v in sd.items()}
    const, mark = reserved(cfg) - 2, reserved(cfg) - 1
    sd["embed"][:, const], sd["embed"][:, mark] = 1.0, 0.0
    sd["embed"][-1, mark] = 4.0
    for i in layers:
        m, p = cfg["layers"][i]["mixer"], f"l{i}."
        H, Dk = m["heads"], m["dim"]
        if cfg["layers"][i]["type"] == LATENT:
            Dr, R = m["rot_dim"], m["kv_rank"]
            sd[p + "mix.dkv.norm"][0] = 1.0
            sd[p + "mix.dkv"][0] = 0.0
            sd[p + "mix.dkv"][0, mark] = 16.0
            for h in range(H):
                q = sd[p + "mix.q"][h * (Dk + Dr):(h + 1) * (Dk + Dr)]
                q *= 0.25
                q[0] = 0.0
                q[0, const] = strength / (0.5 * math.sqrt(R) * m["scale"])
                uk = sd[p + "mix.uk"][h * Dk:(h + 1) * Dk]
                uk[0] = 0.0
                uk[0, 0] = 1.0
        else:  # the norms over the whole projections leave entry 0 of every head near sqrt(dim) in marked keys and in all queries
            for n, rows, col, big in (("q", H, const, 40.0), ("k", m["kv_heads"], mark, 16.0)):
                w = sd[p + "mix." + n]
                for h in range(rows):
                    w[h * Dk] = 0.0
                    w[h * Dk, col] = big
                    sd[p + f"mix.{n}.norm"][h * Dk] = 1.0
    return {k: to_bf16_f32(v) for k, v in sd.items()}
