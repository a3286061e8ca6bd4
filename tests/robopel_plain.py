"""Plain, slow restatement of the Robopel design on the CPU (torch, double precision by default): one
function per mechanism, whole sequences only, no cache and no state. Test infrastructure: it shares
no code with the product and the product never imports it.

Notation: T tokens, W width, H query heads over G key/value heads, D query/key size, E value size.
"""
import math

import torch

from model_files import read_model, write_model  # noqa: F401


# ---------------------------------------------------------------- mechanisms ---
def rms(x, eps, gain=None):
    """x over the root of (mean of squares + eps), then the optional gain."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if gain is None else y * gain


def after_norm(x, y, w, eps):
    """Residual plus the normalised output of a sublayer; the stored weight is the gain's distance from one."""
    return x + rms(y, eps, 1.0 + w)


def min_gru(h, wz, bz, wx, bx, wg, wo, state=None):
    """Gates from the current token only: s' = (1 - z) s + z c, read through silu(wg h)."""
    z = torch.sigmoid(h @ wz.T + bz)
    u = h @ wx.T + bx
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    s = torch.zeros_like(z[0]) if state is None else state
    rows = []
    for t in range(len(h)):
        s = (1 - z[t]) * s + z[t] * cand[t]
        rows.append(s)
    g = h @ wg.T
    return (torch.stack(rows) * (g * torch.sigmoid(g))) @ wo.T


def frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair; long wavelengths slowed down by a factor, with a linear
    transition between two wavelengths."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave, top, bottom = 2 * math.pi / f, scaling["original"] / scaling["high"], scaling["original"] / scaling["low"]
            if wave > bottom:
                f = f / scaling["factor"]
            elif wave >= top:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, freq, first=0):
    """x [T][heads][D]: neighbours (2i, 2i+1) turn by (first + t) freq_i; what follows the pairs passes."""
    T = len(x)
    a = (torch.arange(first, first + T, dtype=x.dtype)[:, None] * torch.tensor(freq, dtype=x.dtype)[None])[:, None, :]
    n = 2 * len(freq)
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y = x.clone()
    y[..., 0:n:2] = u * a.cos() - v * a.sin()
    y[..., 1:n:2] = v * a.cos() + u * a.sin()
    return y


def block_means(k, pool):
    """[T][G][D] -> [T // pool][G][D]: mean of every whole run of `pool` positions."""
    n = len(k) // pool
    return k[: n * pool].reshape(n, pool, *k.shape[1:]).mean(1)


def visible_tokens(T, size):
    i = torch.arange(T)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size) if size else d >= 0


def visible_blocks(T, size, pool):
    """[T][T // pool]: a block whose last position lies outside the window."""
    i, b = torch.arange(T), torch.arange(T // pool)
    return (b[None, :] * pool + pool - 1) <= (i[:, None] - size)


def softcap(x, cap):
    return cap * torch.tanh(x / cap) if cap else x


def sink_attention(q, k, v, scale, cap, size, pool, sink):
    """q [T][H][D], k [T][G][D], v [T][G][E] -> [T][H][E]; tokens of the window and means of the blocks
    before it in one softmax, whose denominator has one more term per head."""
    T, H, _ = q.shape
    keys, vals, see = k, v, visible_tokens(T, size)
    if pool:
        keys, vals = torch.cat([k, block_means(k, pool)]), torch.cat([v, block_means(v, pool)])
        see = torch.cat([see, visible_blocks(T, size, pool)], 1)
    rep = H // k.shape[1]
    s = softcap(torch.einsum("ihd,jhd->hij", q, keys.repeat_interleave(rep, 1)) * scale, cap)
    s = s.masked_fill(~see[None], -math.inf)
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(H, T, 1)], 2)
    p = torch.softmax(s, -1)[..., : len(keys)]
    return torch.einsum("hij,jhe->ihe", p, vals.repeat_interleave(rep, 1))


def poly_norm(z, coef, eps):
    """coef = (a, b, c, e): a n(z) + b n(z^2) + c n(z^3) + e with n the division by the root mean square."""
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def route(h, w, correction, top):
    """(chosen [T][top], their weights [T][top]): chosen by corrected scores, weighted by the scores themselves."""
    s = torch.softmax(h @ w.T, -1)
    idx = torch.topk(s + correction, top, -1).indices
    return idx, s.gather(-1, idx)


def choice_margin(h, w, correction, top):
    """[T]: by how much the last chosen score beats the first one left out."""
    c = torch.softmax(h @ w.T, -1) + correction
    if top == c.shape[-1]:
        return torch.full(c.shape[:1], math.inf, dtype=c.dtype)
    v = torch.topk(c, top + 1, -1).values
    return v[:, top - 1] - v[:, top]


def relu2_expert(h, up, down):
    return torch.relu(h @ up.T).square() @ down.T


def mixture(h, router, correction, top, experts):
    """experts: list of (up, down); router outputs past them are identities."""
    idx, wt = route(h, router, correction, top)
    out = []
    for t in range(len(h)):
        y = torch.zeros_like(h[t])
        for e, a in zip(idx[t].tolist(), wt[t]):
            y = y + a * (relu2_expert(h[t], *experts[e]) if e < len(experts) else h[t])
        out.append(y)
    return torch.stack(out)


# --------------------------------------------------------------------- model ---
class Plain:
    def __init__(self, config, weights, dtype=torch.float64):
        self.c, self.dtype = config, dtype
        self.w = {k: v.to(dtype) for k, v in weights.items()}

    def attention(self, i, h, kv):
        m, p, w, eps = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.w, self.c["norm"]["eps"]
        T, H, G, D, E = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        rot = m.get("rot")
        freq = frequencies(rot["dims"], rot["base"], rot.get("scaling")) if rot else []
        q = rotate(rms((h @ w[p + "q"].T).reshape(T, H, D), eps, w[p + "q.norm"]), freq)
        src = m.get("kv_from")
        if src is None:
            k = rotate(rms((h @ w[p + "k"].T).reshape(T, G, D), eps, w[p + "k.norm"]), freq)
            kv[i] = (k, (h @ w[p + "v"].T).reshape(T, G, E))
        k, v = kv[i if src is None else src]
        y = sink_attention(q, k, v, m["scale"], m.get("softcap"), m["mask"]["size"], m["mask"].get("pool"), w[p + "sink"])
        return (y.reshape(T, H * E) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mixer(self, i, h, kv):
        if self.c["layers"][i]["type"] == "attention":
            return self.attention(i, h, kv)
        w, p = self.w, f"l{i}.mix."
        return min_gru(h, w[p + "z"], w[p + "z.b"], w[p + "x"], w[p + "x.b"], w[p + "g"], w[p + "o"])

    def feed_forward(self, i, h):
        f, p, w = self.c["layers"][i]["mlp"], f"l{i}.mlp.", self.w
        if f["kind"] == "dense":
            return poly_norm(h @ w[p + "up"].T, w[p + "act"], self.c["norm"]["eps"]) @ w[p + "down"].T
        r = f["router"]
        self.margin = torch.minimum(self.margin, choice_margin(h, w[p + "router"], w[p + "correction"], r["top"]))
        return mixture(h, w[p + "router"], w[p + "correction"], r["top"], [(w[p + f"e{e}.up"], w[p + f"e{e}.down"]) for e in range(r["experts"])])

    def forward(self, tokens, want_layers=False):
        c, w, eps = self.c, self.w, self.c["norm"]["eps"]
        x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)] * c["embedding"]["scale"]
        layers, kv = [], {}
        self.margin = torch.full((len(x),), math.inf, dtype=x.dtype)   # per token, over the layers of the last call
        for i, ly in enumerate(c["layers"]):
            x = after_norm(x, self.mixer(i, x, kv), w[f"l{i}.norm1"], eps)
            if ly["mlp"] is not None:
                x = after_norm(x, self.feed_forward(i, x), w[f"l{i}.norm2"], eps)
            layers.append(x)
        lg = rms(x, eps, 1.0 + w["final.norm"]) @ w["head"].T
        return (lg, torch.stack(layers)) if want_layers else lg

    def greedy(self, prompt, n):
        ids, out = list(prompt), []
        for _ in range(n):
            out.append(int(self.forward(ids)[-1].argmax()))
            ids.append(out[-1])
        return out


# ------------------------------------------------- random models and files ---
def make_config(width=48, vocab=96, eps=1e-5, embed_scale=3.0, layers=None):
    return {"architecture": "Robopel", "embedding": {"scale": embed_scale}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def rot(dims=16, base=100.0, scaling=(8.0, 1.0, 4.0, 64)):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(experts, identity, top, ff):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, size=20, pool=6, turn=rot(), scale=0.6, softcap=9.0, kv_from=None, mlp=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": size}, "scale": scale, "vdim": vdim}
    if pool:
        m["mask"]["pool"] = pool
    if turn:
        m["rot"] = turn
    if softcap:
        m["softcap"] = softcap
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mingru(width=56, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def tensor_shapes(c):
    W = c["width"]
    sh = {"embed": (c["vocab"], W)}
    for i, ly in enumerate(c["layers"]):
        m, p, f = ly["mixer"], f"l{i}.", ly["mlp"]
        sh[p + "norm1"] = (W,)
        if ly["type"] == "mingru":
            K = m["width"]
            sh.update({p + "mix.z": (K, W), p + "mix.x": (K, W), p + "mix.g": (K, W), p + "mix.z.b": (K,), p + "mix.x.b": (K,), p + "mix.o": (W, K)})
        else:
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            sh.update({p + "mix.q": (H * D, W), p + "mix.q.norm": (D,), p + "mix.sink": (H,), p + "mix.g": (H * E, W), p + "mix.o": (W, H * E)})
            if "kv_from" not in m:
                sh.update({p + "mix.k": (G * D, W), p + "mix.v": (G * E, W), p + "mix.k.norm": (D,)})
        if f is None:
            continue
        sh[p + "norm2"] = (W,)
        if f["kind"] == "dense":
            sh.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"]), p + "mlp.act": (4,)})
        else:
            n = f["router"]["experts"] + f["router"]["identity"]
            sh.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            for e in range(f["router"]["experts"]):
                sh.update({p + f"mlp.e{e}.up": (f["expert"]["ff"], W), p + f"mlp.e{e}.down": (W, f["expert"]["ff"])})
    sh.update({"final.norm": (W,), "head": (c["vocab"], W)})
    return sh


def make_weights(c, seed=0):
    """Seeded bf16 weights with every mechanism well away from its neutral value: queries long enough for
    single keys to stand out, sinks of the size of the scores, recurrences that remember for long."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for n, s in tensor_shapes(c).items():
        r = torch.randn(s, generator=g)
        leaf = n.split(".", 1)[-1]
        if leaf in ("norm1", "norm2") or n == "final.norm":
            v = 0.25 * r
        elif leaf == "mix.q.norm":
            v = 1.8 + 0.2 * r
        elif leaf == "mix.k.norm":
            v = 1.0 + 0.2 * r
        elif leaf == "mix.sink":
            v = 2.0 + r
        elif leaf == "mix.z.b":
            v = -2.0 + r
        elif leaf == "mix.x.b":
            v = 0.3 * r
        elif leaf == "mlp.act":
            v = torch.tensor([0.7, -0.5, 0.4, 0.3]) + 0.1 * r
        elif leaf == "mlp.router":
            v = 1.5 * r / math.sqrt(s[1])
        elif leaf == "mlp.correction":
            v = 0.4 * r
        elif n == "embed":
            v = 0.5 * r
        else:
            v = r / math.sqrt(s[1])
        out[n] = v.to(torch.bfloat16)
    return out


def steady_tokens(plain, n, seed, margin=0.03, block=3):
    """n random tokens whose expert choices are not close calls."""
    g = torch.Generator().manual_seed(seed)
    ids = []
    while len(ids) < n:
        for _ in range(60):
            more = torch.randint(0, plain.c["vocab"], (min(block, n - len(ids)),), generator=g).tolist()
            plain.forward(ids + more)
            if plain.margin[len(ids):].min() > margin:
                break
        ids += more
    return ids
