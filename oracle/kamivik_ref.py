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

    def forward(self, tokens, st=None, taps=None):
        """tokens -> logits [T, vocab]; st is updated in place.  taps (a list) receives the stream after every layer."""
        cfg, sd = self.cfg, self.sd
        st = self.new_state() if st is None else st
        pos = np.arange(st["pos"], st["pos"] + len(tokens))
        x = sd["embed"][np.asarray(tokens)]
        for i, ly in enumerate(cfg["layers"]):
            h = rms_norm(x, sd[f"l{i}.norm1"], self.eps)
            y = self.mixer(i, ly, h, st, pos) * sd[f"l{i}.ls1"]
            if ly.get("mlp") is not None:
                y = y + mixture(h, self.sub(f"l{i}.mlp."), ly["mlp"]) * sd[f"l{i}.ls2"]
            x = x + cfg["residual_mult"] * y
            if taps is not None:
                taps.append(x.copy())
        st["pos"] += len(tokens)
        return rms_norm(x, sd["final.norm"], self.eps) @ sd["head"].T
