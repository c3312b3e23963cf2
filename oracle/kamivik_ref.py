"""Plain, slow float64 restatement of the Kamivik decoder (numpy only; one function per mechanism).

The design: layers whose two sublayers read ONE normed copy of the stream and are added together through per-channel gains and
a common factor, x <- x + m (a * mixer(h) + b * ff(h)), h = norm(x); mixers that attend over a cached low-rank latent and one
rotated key part shared by all heads (queries projected directly from h, interleaved rotation, no softmax sink) — either over
every earlier position with one output gate per head, or over a sliding window with a gate per output entry; mixtures of
ungated erf-GELU experts whose router adds a bias to its logits and takes a softmax over the chosen ones.  Notation: T tokens,
W width, H heads, Dk / Dr / Dv unrotated / rotated / value sizes per head, R latent rank.  Nothing here is shared with the CUDA
path; the GPU tests compare the engine against these functions.
"""
import math

import numpy as np

F = np.float64
_erf = np.vectorize(math.erf, otypes=[F])


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    x = np.asarray(x, F)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * np.asarray(w, F)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def rotate_interleaved(v, pos, base, dims):
    """Rotate the first `dims` entries of the last axis: entries 2i and 2i + 1 form a pair, angle pos * base^(-2i/dims)."""
    v = np.array(v, F)
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=F) / dims)
    a = np.asarray(pos, F)[..., None] * f
    c, s = np.cos(a), np.sin(a)
    while c.ndim < v.ndim:  # head axes between the token axis and the last axis
        c, s = c[..., None, :], s[..., None, :]
    u, w = v[..., 0:dims:2].copy(), v[..., 1:dims:2].copy()
    v[..., 0:dims:2] = u * c - w * s
    v[..., 1:dims:2] = w * c + u * s
    return v


# ------------------------------------------------------------------ latent attention
def latent_row(h, p, m, pos):
    """What is kept per token: the normed latent [T, R] and the rotated shared key part [T, Dr]."""
    R = m["kv_rank"]
    d = h @ p["dkv"].T
    return rms_norm(d[:, :R], p["dkv.norm"], m["eps"]), rotate_interleaved(d[:, R:], pos, m["rot"]["base"], m["rot"]["dims"])


def visible(pos, kpos, window):
    """[T, J] mask: key positions each query position sees (window None: every earlier one)."""
    dist = np.asarray(pos)[:, None] - np.asarray(kpos)[None, :]
    return (dist >= 0) if window is None else (dist >= 0) & (dist < window)


def softmax_seen(s, seen):
    """softmax over the last axis of s [T, H, J] restricted to seen [T, J]"""
    s = np.where(seen[:, None, :], s, -np.inf)
    e = np.exp(s - s.max(-1, keepdims=True))
    return e / e.sum(-1, keepdims=True)


def latent_heads(h, p, m, pos, c, kr, kpos):
    """Head outputs [T, H, Dv]; c / kr / kpos: rows and positions of EVERY key so far (this call's tokens included)."""
    T = h.shape[0]
    H, Dk, Dr, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ p["q"].T).reshape(T, H, Dk + Dr)
    qn, qr = q[:, :, :Dk], rotate_interleaved(q[:, :, Dk:], pos, m["rot"]["base"], m["rot"]["dims"])
    kn = (c @ p["uk"].T).reshape(-1, H, Dk)
    val = (c @ p["uv"].T).reshape(-1, H, Dv)
    s = (np.einsum("thd,jhd->thj", qn, kn) + np.einsum("thd,jd->thj", qr, kr)) * m["scale"]
    mask = m.get("mask")
    w = softmax_seen(s, visible(pos, kpos, mask["size"] if mask else None))
    return np.einsum("thj,jhv->thv", w, val)


def gate_heads(o, h, g):
    """one gate per head: o [T, H, Dv], g [H, W]"""
    return o * sigmoid(h @ g.T)[:, :, None]


def gate_entries(o, h, g):
    """one gate per entry of the concatenated heads: g [H * Dv, W]"""
    return o * sigmoid(h @ g.T).reshape(o.shape)


# ------------------------------------------------------------------ mixture of experts
def route(h, router, bias, top):
    """chosen experts [T, top] (largest biased logits first) and the softmax over their logits"""
    z = h @ router.T + bias
    ids = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, ids, -1)
    e = np.exp(zc - zc.max(-1, keepdims=True))
    return ids, e / e.sum(-1, keepdims=True)


def route_margin(h, router, bias, top):
    """how far the last chosen biased logit lies above the best one left out (inf when all are chosen), per token"""
    z = -np.sort(-(h @ router.T + bias), axis=-1)
    return z[:, top - 1] - z[:, top] if z.shape[1] > top else np.full(len(z), np.inf)


def expert(h, up, down):
    return gelu_erf(h @ up.T) @ down.T


def mixture(h, p, mlp):
    r = mlp["router"]
    ids, w = route(h, p["router"], p["router.b"], r["top"])
    out = np.zeros((h.shape[0], p["e0.down"].shape[0]), F)
    for e in range(r["experts"]):
        t, k = np.nonzero(ids == e)
        if len(t):
            np.add.at(out, t, w[t, k][:, None] * expert(h[t], p[f"e{e}.up"], p[f"e{e}.down"]))
    return out


# ------------------------------------------------------------------ the model
class KamivikOracle:
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
        return {"pos": 0, "rows": {}}

    def mixer(self, i, ly, h, st, pos):
        m = dict(ly["mixer"], eps=self.eps)
        if ly["type"] == "latent_attention":
            m.pop("mask", None)
        p = self.sub(f"l{i}.mix.")
        c, kr = latent_row(h, p, m, pos)
        if i in st["rows"]:
            pc, pr = st["rows"][i]
            c, kr = np.concatenate([pc, c]), np.concatenate([pr, kr])
        st["rows"][i] = (c, kr)
        o = latent_heads(h, p, m, pos, c, kr, np.arange(c.shape[0]))
        o = gate_heads(o, h, p["g"]) if ly["type"] == "latent_attention" else gate_entries(o, h, p["g"])
        return o.reshape(h.shape[0], -1) @ p["o"].T

    def forward(self, tokens, st=None, taps=None, margins=None):
        """tokens -> logits [T, vocab]; st is updated in place.  taps / margins (lists) receive the stream after every layer /
        every router's margins."""
        cfg, sd = self.cfg, self.sd
        st = self.new_state() if st is None else st
        pos = np.arange(st["pos"], st["pos"] + len(tokens))
        x = sd["embed"][np.asarray(tokens)]
        for i, ly in enumerate(cfg["layers"]):
            h = rms_norm(x, sd[f"l{i}.norm1"], self.eps)
            y = self.mixer(i, ly, h, st, pos) * sd[f"l{i}.ls1"]
            if ly.get("mlp") is not None:
                if margins is not None:
                    margins.append(route_margin(h, sd[f"l{i}.mlp.router"], sd[f"l{i}.mlp.router.b"], ly["mlp"]["router"]["top"]))
                y = y + mixture(h, self.sub(f"l{i}.mlp."), ly["mlp"]) * sd[f"l{i}.ls2"]
            x = x + cfg["residual_mult"] * y
            if taps is not None:
                taps.append(x.copy())
        st["pos"] += len(tokens)
        return rms_norm(x, sd["final.norm"], self.eps) @ sd["head"].T


# ------------------------------------------------------------------ random checkpoints for tests
FULL, WIN = "latent_attention", "latent_attention_2"


def mixer_cfg(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, base=1000.0, window=None, scale=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, rot=dict(dims=rot_dim, base=float(base)),
             scale=float(scale if scale is not None else (dim + rot_dim) ** -0.5))
    if window:
        m["mask"] = dict(size=window)
    return m


def random_config(width=96, vocab=120, order=((FULL, True), (WIN, True), (FULL, False)), full=None, win=None, window=37, experts=6, top=2, ff=40,
                  mult=0.8, eps=1e-5, per_layer=None, per_mlp=None):
    """order: (type, has a feed-forward) per layer; per_layer / per_mlp {i: dict}: that layer's mixer / feed-forward."""
    layers = []
    for i, (kind, has_ff) in enumerate(order):
        mixer = dict(full or mixer_cfg()) if kind == FULL else dict(win or mixer_cfg(heads=4, dim=24, rot_dim=16, vdim=16, kv_rank=48, base=300.0))
        if kind == WIN and "mask" not in mixer:
            mixer["mask"] = dict(size=window)
        if per_layer and i in per_layer:
            mixer = per_layer[i]
        mlp = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top)) if has_ff else None
        if per_mlp and i in per_mlp:
            mlp = per_mlp[i]
        layers.append(dict(type=kind, mixer=mixer, mlp=mlp))
    return dict(architecture="Kamivik", width=width, vocab=vocab, layers=layers, norm=dict(eps=eps), residual_mult=float(mult))


def reserved(cfg):
    """leading stream entries that no sublayer writes (their gains are zero): one per expert, then two for planted features"""
    return max([ly["mlp"]["router"]["experts"] for ly in cfg["layers"] if ly["mlp"]] + [0]) + 2


def random_state_dict(cfg, seed=0):
    """Router choices are made by the leading stream entries, which hold a shuffled grid of values per token and stay as
    embedded, so that no choice is a close call; everything else is random."""
    from .weights import _rng, _t, to_bf16_f32
    W, V = cfg["width"], cfg["vocab"]
    s = lambda n: 1.0 / math.sqrt(n)
    n_res = reserved(cfg)
    E0 = n_res - 2
    embed = _t(seed, "embed", (V, W), 0.5)
    g = _rng(seed, "grid")
    for v in range(V):
        embed[v, :E0] = (g.permutation(E0) - (E0 - 1) / 2.0) * min(0.5, 4.0 / max(E0, 1))
    embed[:, E0:n_res] = 0.0
    sd = {"embed": to_bf16_f32(embed), "final.norm": _t(seed, "fn", (W,), 0.1, 1.0), "head": _t(seed, "head", (V, W), s(W))}
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}."
        H, Dk, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        sd[p + "norm1"] = _t(seed, p + "n1", (W,), 0.1, 1.0)
        sd[p + "norm1"][:n_res] = 1.0
        sd[p + "mix.q"] = _t(seed, p + "q", (H * (Dk + Dr), W), 1.5 * s(W))
        sd[p + "mix.dkv"] = _t(seed, p + "dkv", (R + Dr, W), 1.5 * s(W))
        sd[p + "mix.dkv.norm"] = _t(seed, p + "dkvn", (R,), 0.1, 1.0)
        sd[p + "mix.uk"] = _t(seed, p + "uk", (H * Dk, R), 1.5 * s(R))
        sd[p + "mix.uv"] = _t(seed, p + "uv", (H * Dv, R), 1.5 * s(R))
        sd[p + "mix.g"] = _t(seed, p + "g", (H if ly["type"] == FULL else H * Dv, W), 1.5 * s(W))
        sd[p + "mix.o"] = _t(seed, p + "o", (W, H * Dv), 2.0 * s(H * Dv))
        for n in ("ls1", "ls2"):
            gain = _t(seed, p + n, (W,), 0.2, 0.8)
            gain[:n_res] = 0.0
            if n == "ls1" or ly["mlp"]:
                sd[p + n] = gain
        if ly["mlp"]:
            E, Fn = ly["mlp"]["router"]["experts"], ly["mlp"]["expert"]["ff"]
            router = _t(seed, p + "router", (E, W), (0.3 if E0 <= 12 else 0.1) * s(W))
            router[:, :n_res] = 0.0
            for e in range(E):
                router[e, e] = 8.0 / min(0.5, 4.0 / E0) * 0.5
            sd[p + "mlp.router"] = to_bf16_f32(router)
            sd[p + "mlp.router.b"] = _t(seed, p + "rb", (E,), 0.2)
            for e in range(E):
                sd[p + f"mlp.e{e}.up"] = _t(seed, p + f"e{e}u", (Fn, W), 2.0 * s(W))
                sd[p + f"mlp.e{e}.down"] = _t(seed, p + f"e{e}d", (W, Fn), 2.0 * s(Fn))
    return sd


def plant_marker(cfg, sd, layers, strength=14.0):
    """Token vocab - 1 becomes a marker: in the named layers every head's score for it stands out by `strength` wherever it is
    seen, and its latent is unlike any other token's, so whether a position sees it shows in the logits."""
    sd = {k: v.copy() for k, v in sd.items()}
    const, mark = reserved(cfg) - 2, reserved(cfg) - 1
    sd["embed"][:, const], sd["embed"][:, mark] = 1.0, 0.0
    sd["embed"][-1, mark] = 4.0
    for i in layers:
        m, p = cfg["layers"][i]["mixer"], f"l{i}."
        H, Dk, Dr, R = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
        sd[p + "mix.dkv.norm"][0] = 1.0
        sd[p + "mix.dkv"][0] = 0.0
        sd[p + "mix.dkv"][0, mark] = 16.0
        for h in range(H):
            q = sd[p + "mix.q"][h * (Dk + Dr):(h + 1) * (Dk + Dr)]
            q *= 0.25
            q[0] = 0.0
            q[0, const] = float(np.float32(strength / (0.5 * math.sqrt(R) * m["scale"])))
            uk = sd[p + "mix.uk"][h * Dk:(h + 1) * Dk]
            uk[0] = 0.0
            uk[0, 0] = 1.0
    from .weights import to_bf16_f32
    return {k: to_bf16_f32(v) for k, v in sd.items()}
