"""Plain, slow restatement of the Sinepel design on the CPU (torch, double precision by default):
one function per mechanism, whole sequences only, no cache and no state. Test infrastructure: it
shares no code with the product and the product never imports it.

Notation: T tokens, W width, S residual streams, H query heads over G key heads of size D.
"""
import math

import torch

from model_files import read_model, write_model  # noqa: F401


# ---------------------------------------------------------------- mechanisms ---
def rms(x, eps, w=None):
    """x / sqrt(mean(x^2) + eps), then the optional gain."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def embed(tokens, table, scale, pos_table):
    """Scaled token rows plus the learned vector of each position (unscaled)."""
    return table[tokens] * scale + pos_table[: len(tokens)]


def streams_read(x, w_in):
    """Weighted sum of the streams: x [T][S][W], w_in [S] -> [T][W]."""
    return torch.einsum("tsw,s->tw", x, w_in)


def streams_write(x, mix, w_out, y):
    """Every stream t from all old streams s: sum_s mix[s][t] x_s + w_out[t] y."""
    return torch.einsum("tsw,su->tuw", x, mix) + w_out[None, :, None] * y[:, None, :]


def token_shift(h, amount):
    """h + (h of the previous token - h) * amount; the first token's predecessor is zero."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * amount


def short_conv(u, taps):
    """Causal convolution per channel: u [T][C], taps [C][J]; the last tap meets the current token."""
    J = taps.shape[1]
    y = torch.zeros_like(u)
    for j in range(J):
        back = J - 1 - j
        shifted = torch.cat([torch.zeros_like(u[:back]), u[: len(u) - back]]) if back else u
        y = y + shifted[: len(u)] * taps[:, j]
    return y


def visible(T, chunk):
    """[i][j] true where j <= i and both lie in the same chunk of positions."""
    i = torch.arange(T)
    m = i[:, None] >= i[None, :]
    if chunk:
        m &= (i[:, None] // chunk) == (i[None, :] // chunk)
    return m


def log_distance(T, r1, r2):
    """[H][i][j]: r1_h ln(1 + r2_h (i - j)) for j <= i (0 above the diagonal)."""
    i = torch.arange(T)
    d = (i[:, None] - i[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log1p(r2[:, None, None] * d)


def shared_kv_attention(q, k, scale, temp, r1, r2, chunk):
    """q [T][H][D], k [T][G][D]; the keys are also the values. Returns [T][H][D]."""
    T, H, _ = q.shape
    kk = k.repeat_interleave(H // k.shape[1], dim=1)
    s = torch.einsum("ihd,jhd->hij", q, kk) * scale * temp[:, None, None] - log_distance(T, r1, r2)
    s = s.masked_fill(~visible(T, chunk)[None], -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), kk)


def relu2_mlp(h, up, down):
    return torch.relu(h @ up.T).square() @ down.T


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


# --------------------------------------------------------------------- model ---
class Plain:
    def __init__(self, config, weights, dtype=torch.float64):
        self.c, self.dtype = config, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}

    def mixer(self, i, h):
        m, p, w = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.w
        T, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
        q = short_conv(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.conv"])
        k = short_conv(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.conv"])
        y = shared_kv_attention(q.reshape(T, H, D), k.reshape(T, G, D), m["scale"], w[p + "temp"], w[p + "r1"], w[p + "r2"],
                                m["mask"]["size"])
        return y.reshape(T, H * D) @ w[p + "o"].T

    def sublayer(self, x, i, q, norm, f):
        w, p = self.w, f"l{i}.hc{q}."
        h = rms(streams_read(x, w[p + "in"]), self.c["norm"]["eps"], w[f"l{i}.{norm}"])
        return streams_write(x, w[p + "mix"], w[p + "out"], f(h))

    def forward(self, tokens, want_layers=False):
        c, w = self.c, self.w
        t = torch.as_tensor(list(tokens), dtype=torch.long)
        x = embed(t, w["embed"], c["embedding"]["scale"], w["pos"])[:, None, :].repeat(1, c["streams"], 1)
        layers = []
        for i, ly in enumerate(c["layers"]):
            x = self.sublayer(x, i, 1, "norm1", lambda h: self.mixer(i, token_shift(h, w[f"l{i}.shift"])))
            if ly["mlp"] is not None:
                x = self.sublayer(x, i, 2, "norm2", lambda h: relu2_mlp(h, w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"]))
            layers.append(x.sum(1))
        h = rms(x.sum(1), c["norm"]["eps"], w["final.norm"])
        lg = softcap(h @ w["head"].T, c["logit_softcap"])
        return (lg, torch.stack(layers)) if want_layers else lg

    def greedy(self, prompt, n):
        ids, out = list(prompt), []
        for _ in range(n):
            out.append(int(self.forward(ids)[-1].argmax()))
            ids.append(out[-1])
        return out


# ------------------------------------------------- random models and files ---
def make_config(width=48, vocab=96, streams=3, max_positions=512, eps=1e-5, embed_scale=3.0, cap=20.0, layers=None):
    return {"architecture": "Sinepel", "embedding": {"scale": embed_scale}, "layers": layers, "logit_softcap": cap,
            "max_positions": max_positions, "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


def make_layer(heads=4, kv_heads=2, dim=16, conv=3, chunk=24, scale=0.3, ff=80):
    return {"type": "attention", "mixer": {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": chunk},
                                           "scale": scale, "vdim": dim},
            "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def tensor_shapes(c):
    W, S, V = c["width"], c["streams"], c["vocab"]
    sh = {"embed": (V, W), "pos": (c["max_positions"], W)}
    for i, ly in enumerate(c["layers"]):
        m, p = ly["mixer"], f"l{i}."
        Q, K = m["heads"] * m["dim"], m["kv_heads"] * m["dim"]
        sh.update({p + "norm1": (W,), p + "shift": (W,), p + "mix.q": (Q, W), p + "mix.q.b": (Q,), p + "mix.k": (K, W), p + "mix.k.b": (K,),
                   p + "mix.q.conv": (Q, m["conv"]), p + "mix.k.conv": (K, m["conv"]), p + "mix.r1": (m["heads"],), p + "mix.r2": (m["heads"],),
                   p + "mix.temp": (m["heads"],), p + "mix.o": (W, Q), p + "hc1.in": (S,), p + "hc1.out": (S,), p + "hc1.mix": (S, S)})
        if ly["mlp"] is not None:
            F = ly["mlp"]["ff"]
            sh.update({p + "norm2": (W,), p + "mlp.up": (F, W), p + "mlp.down": (W, F), p + "hc2.in": (S,), p + "hc2.out": (S,),
                       p + "hc2.mix": (S, S)})
    sh.update({"final.norm": (W,), "head": (V, W)})
    return sh


def make_weights(c, seed=0):
    """Seeded bf16 weights with every mechanism well away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in tensor_shapes(c).items():
        r = torch.randn(s, generator=g)
        leaf = n.split(".", 1)[-1]
        if leaf.startswith("norm") or n == "final.norm":
            v = 1.0 + 0.2 * r
        elif leaf == "shift":
            v = torch.rand(s, generator=g)
        elif leaf.endswith(".b"):
            v = 0.3 * r
        elif leaf.endswith(".conv"):
            v = 0.3 * r
            v[:, -1] += 0.8
        elif leaf in ("mix.r1", "mix.r2"):
            v = torch.rand(s, generator=g) + 0.2
        elif leaf == "mix.temp":
            v = 0.6 + torch.rand(s, generator=g)
        elif leaf.endswith(".in"):
            v = 1.0 / s[0] + 0.3 * r
        elif leaf.startswith("hc") and leaf.endswith(".out"):
            v = 0.7 + 0.3 * r
        elif leaf.startswith("hc") and leaf.endswith(".mix"):
            v = 0.8 * torch.eye(s[0]) + 0.15 * r
        elif n in ("embed", "pos"):
            v = 0.5 * r
        else:
            v = r / math.sqrt(s[1])
        out[n] = v.to(torch.bfloat16)
    return out
