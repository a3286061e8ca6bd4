"""Prefill and decode throughput of architectures with a row engine (bench.py --design), on random
weights at sizes that resemble a real model's layers, beside the framework's closest other model at equal
width: the INT4 hybrid beside Sinepel, Sinepel beside Robopel. Times are device events around whole calls
of the public API after warm-up. A step streams more than L2 holds from width 2048 on; at width 1024
(about 110 MB) part of it stays there."""
import json
import os
import tempfile

import numpy as np

# name -> (width, heads, kv_heads, dim, ff, layers, vocab, chunk, preset of the INT4 hybrid of that width, depth and vocabulary)
SIZES = {
    "w1024": (1024, 8, 2, 128, 4096, 2, 32000, 1024, "mini"),
    "w2048": (2048, 16, 4, 128, 8192, 4, 32000, 2048, "small"),
    "w4096": (4096, 32, 8, 128, 14336, 4, 32000, 2048, None),
}
STREAMS, TAPS = 4, 4
# Robopel at the same widths, heads, feed-forward, depth and vocabulary, its window half of the chunk and
# block means before it: attention with a dense feed-forward and recurrences with a mixture take turns, the
# second attention reads the first one's cache. name -> (experts, identities, chosen, expert ff)
MIXTURES = {"w1024": (16, 2, 2, 1024), "w2048": (32, 2, 4, 1024), "w4096": (32, 2, 4, 2048)}
POOL = 16


class Sinepel:
    @staticmethod
    def config(name):
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        layer = {"type": "attention", "mixer": {"conv": TAPS, "dim": D, "heads": H, "kv_heads": G, "mask": {"size": chunk}, "scale": D ** -0.5, "vdim": D},
                 "mlp": {"ff": F, "kind": "dense"}}
        return {"architecture": "Sinepel", "embedding": {"scale": 1.0}, "layers": [layer] * L, "logit_softcap": 30.0, "max_positions": 8192,
                "norm": {"eps": 1e-6}, "streams": STREAMS, "vocab": V, "width": W}

    @staticmethod
    def step_bytes(name, batch, ctx):
        """Weights and keys that a step of `batch` sequences at a full chunk reads."""
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        return 2 * (L * ((H + G) * D * W + H * D * W + 2 * F * W) + V * W) + batch * L * chunk * G * D * 2

    @staticmethod
    def row_flops(name, prompt):
        """Products per prompt row (without logits), attention at its mean reach."""
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        return 2 * L * ((H + G) * D * W + H * D * W + 2 * F * W) + L * 4 * H * D * chunk / 2


class Robopel:
    @staticmethod
    def config(name):
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        window = chunk // 2
        E, ident, top, Fe = MIXTURES[name]
        layers = []
        for i in range(L):
            if i % 2:
                layers.append({"type": "mingru", "mixer": {"width": W},
                               "mlp": {"expert": {"ff": Fe}, "kind": "moe", "router": {"experts": E, "identity": ident, "top": top}}})
                continue
            m = {"dim": D, "heads": H, "kv_heads": G, "mask": {"pool": POOL, "size": window}, "scale": D ** -0.5, "softcap": 30.0, "vdim": D,
                 "rot": {"base": 10000.0, "dims": D, "scaling": {"factor": 8.0, "high": 4.0, "low": 1.0, "original": 2048}}}
            if i:
                m["kv_from"] = 0
            layers.append({"type": "attention", "mixer": m, "mlp": {"ff": F, "kind": "dense"}})
        return {"architecture": "Robopel", "embedding": {"scale": 1.0}, "layers": layers, "norm": {"eps": 1e-6}, "vocab": V, "width": W}

    @staticmethod
    def _dense(name):
        W, H, G, D, F, L, V, _, _ = SIZES[name]
        E, ident, _, _ = MIXTURES[name]
        att, rec = (L + 1) // 2, L // 2
        return att * (3 * H * D * W + 2 * F * W) + 2 * G * D * W + rec * (4 * W * W + (E + ident) * W)

    @staticmethod
    def step_bytes(name, batch, ctx):
        """Weights (of the experts that a uniform choice touches), keys and values of the window and block means."""
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        window = chunk // 2
        E, ident, top, Fe = MIXTURES[name]
        touched = E * (1 - (1 - top / (E + ident)) ** batch)
        keys = min(ctx, window) + max(0, ctx - window + 1) // POOL
        return 2 * (Robopel._dense(name) + V * W + (L // 2) * touched * 2 * Fe * W) + batch * ((L + 1) // 2) * keys * G * D * 2 * 2

    @staticmethod
    def row_flops(name, prompt):
        W, H, G, D, F, L, V, chunk, _ = SIZES[name]
        window = chunk // 2
        E, ident, top, Fe = MIXTURES[name]
        i = np.arange(prompt)
        reach = (np.minimum(i + 1, window) + np.maximum(0, i - window + 1) // POOL).mean()
        return 2 * (Robopel._dense(name) + (L // 2) * top * E / (E + ident) * 2 * Fe * W) + ((L + 1) // 2) * 4 * H * D * reach


DESIGNS = {"sinepel": Sinepel, "robopel": Robopel}


def open_model(dev, name, seed=0, design="sinepel"):
    from . import runtime
    f = tempfile.NamedTemporaryFile("w", suffix=".json", delete=False)
    json.dump(DESIGNS[design].config(name), f)
    f.close()
    try:
        return runtime.Model(dev, f"synth:config:{f.name}:seed={seed}")
    finally:
        os.unlink(f.name)


def timed(dev, fn, reps, warm=2):
    for _ in range(warm):
        fn()
    dev.sync()
    ms = []
    for _ in range(reps):
        a, b = dev.event(), dev.event()
        a.record()
        fn()
        b.record()
        dev.sync()
        ms.append(a.elapsed_ms(b))
    return float(np.median(ms))


def measure(dev, model, ctx, prompt, batches, steps, flags=0):
    """Decode at a full chunk / long context, prompts, and batched steps of one model."""
    from . import runtime
    V = model.config["vocab"]
    ids = np.random.default_rng(0).integers(0, V, prompt + 8).astype(np.int32)
    out = {}
    s = runtime.Session(model, max(prompt, ctx) + steps + 16, flags)
    ms = timed(dev, lambda: s.prefill(ids[:prompt]), 5)
    out["prefill"] = {"tokens": prompt, "ms": ms, "tokens_per_s": prompt / ms * 1e3}
    s.reset()
    s.prefill(ids[:ctx])
    runs = []
    for _ in range(4):
        _, ms = s.generate(ids[:1], steps, start_pos=ctx, timed=True)
        runs.append(ms / steps)
    out["decode"] = {"context": ctx, "ms_per_token": float(np.median(runs[1:])), "tokens_per_s": 1e3 / float(np.median(runs[1:])),
                     "launches": s.launches_per_token()}
    s.close()
    for B in batches:
        b = runtime.BatchDecode(model, B, ctx + 64)
        b.set_inputs(ids[:B] if B <= len(ids) else np.resize(ids, B), np.full(B, ctx, np.int32))
        ms = timed(dev, b.step, 10, 3)
        out[f"batch{B}"] = {"context": ctx, "ms_per_step": ms, "tokens_per_s": B / ms * 1e3}
        b.close()
    return out


def run(dev, names, hbm_gbs, bf16_tflops, steps=32, design="sinepel"):
    from . import runtime
    prompt = 4096

    def one(name, which):
        ctx = SIZES[name][7] - steps - 24
        m = open_model(dev, name, design=which)
        r = measure(dev, m, ctx, prompt, (16, 64), steps)
        m.close()
        d = DESIGNS[which]
        for x, ms, B in [(r["decode"], r["decode"]["ms_per_token"], 1)] + [(r[f"batch{B}"], r[f"batch{B}"]["ms_per_step"], B) for B in (16, 64)]:
            x["gbs"] = d.step_bytes(name, B, ctx) / ms / 1e6
            x["of_hbm"] = x["gbs"] / hbm_gbs
        r["prefill"]["tflops"] = d.row_flops(name, prompt) * prompt / r["prefill"]["ms"] / 1e9
        r["prefill"]["of_bf16"] = r["prefill"]["tflops"] / bf16_tflops
        return r
    rows = {}
    for name in names:
        rows[name] = {design: one(name, design)}
        preset = SIZES[name][8]
        if design == "robopel":
            rows[name]["sinepel"] = one(name, "sinepel")
        elif preset:
            m = runtime.Model(dev, f"synth:{preset}:seed=0")
            rows[name]["int4_hybrid_" + preset] = measure(dev, m, SIZES[name][7] - steps - 24, prompt, (16, 64), steps, runtime.Session.PERSISTENT)
            m.close()
    return rows


def once(name, what, design="sinepel"):
    """A few launches to capture: a prompt pass of 2048 rows, four decode steps at position 2000, or two
    batched steps (what = the batch) at position 2000."""
    from . import cuda_abi, runtime
    dev = cuda_abi.Device(0)
    m = open_model(dev, name, design=design)
    ids = np.random.default_rng(0).integers(0, m.config["vocab"], 4096).astype(np.int32)
    dev.sync()
    if what == "prefill":
        s = runtime.Session(m, 4096)
        s.prefill(ids[:2048])
    elif what == "decode":
        s = runtime.Session(m, 4096)
        s.generate(ids[:1], 4, start_pos=2000)
    else:
        s = runtime.BatchDecode(m, int(what), 2100)
        s.set_inputs(ids[:int(what)], np.full(int(what), 2000, np.int32))
        s.step()
        s.step()
    dev.sync()
    s.close()
    m.close()
    dev.close()


if __name__ == "__main__":
    import argparse
    ap = argparse.ArgumentParser(description=once.__doc__)
    ap.add_argument("size", choices=sorted(SIZES))
    ap.add_argument("what", help="prefill, decode or a batch size")
    ap.add_argument("--design", choices=sorted(DESIGNS), default="sinepel")
    a = ap.parse_args()
    once(a.size, a.what, a.design)
