"""Prefill and decode throughput of architectures with a row engine (bench.py --design), on random
weights at sizes that resemble a real model's layers, beside the INT4 hybrid at equal width, depth and
vocabulary. Times are device events around whole calls of the public API after warm-up. A step
streams more than L2 holds from width 2048 on; at width 1024 (about 110 MB) part of it stays there."""
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


def config(name):
    W, H, G, D, F, L, V, chunk, _ = SIZES[name]
    layer = {"type": "attention", "mixer": {"conv": TAPS, "dim": D, "heads": H, "kv_heads": G, "mask": {"size": chunk}, "scale": D ** -0.5, "vdim": D},
             "mlp": {"ff": F, "kind": "dense"}}
    return {"architecture": "Sinepel", "embedding": {"scale": 1.0}, "layers": [layer] * L, "logit_softcap": 30.0, "max_positions": 8192,
            "norm": {"eps": 1e-6}, "streams": STREAMS, "vocab": V, "width": W}


def costs(name):
    """Per token: weight bytes of a decode step, products of a prompt row (without logits), stream bytes."""
    W, H, G, D, F, L, V, chunk, _ = SIZES[name]
    mats = L * ((H + G) * D * W + H * D * W + 2 * F * W)
    return {"weight_bytes": 2 * (mats + V * W), "key_bytes_full_chunk": L * chunk * G * D * 2, "matrix_flops_per_row": 2 * mats,
            "attention_flops_per_row_mean": L * 4 * H * D * chunk / 2}


def open_model(dev, name, seed=0):
    from . import runtime
    f = tempfile.NamedTemporaryFile("w", suffix=".json", delete=False)
    json.dump(config(name), f)
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


def run(dev, names, hbm_gbs, bf16_tflops, steps=32):
    from . import runtime
    rows = {}
    for name in names:
        W, H, G, D, F, L, V, chunk, preset = SIZES[name]
        ctx, prompt = chunk - steps - 24, 4096
        m = open_model(dev, name)
        r = measure(dev, m, ctx, prompt, (16, 64), steps)
        m.close()
        c = costs(name)
        by = c["weight_bytes"] + c["key_bytes_full_chunk"]
        r["decode"]["gbs"] = by / r["decode"]["ms_per_token"] / 1e6
        r["decode"]["of_hbm"] = r["decode"]["gbs"] / hbm_gbs
        fl = (c["matrix_flops_per_row"] + c["attention_flops_per_row_mean"]) * prompt
        r["prefill"]["tflops"] = fl / r["prefill"]["ms"] / 1e9
        r["prefill"]["of_bf16"] = r["prefill"]["tflops"] / bf16_tflops
        for B in (16, 64):
            x = r[f"batch{B}"]
            x["gbs"] = (c["weight_bytes"] + B * c["key_bytes_full_chunk"]) / x["ms_per_step"] / 1e6
            x["of_hbm"] = x["gbs"] / hbm_gbs
        rows[name] = {"sinepel": r}
        if preset:
            m = runtime.Model(dev, f"synth:{preset}:seed=0")
            rows[name]["int4_hybrid_" + preset] = measure(dev, m, ctx, min(prompt, 4096), (16, 64), steps, runtime.Session.PERSISTENT)
            m.close()
    return rows


def once(name, what):
    """A few launches to capture: a prompt pass of 2048 rows, four decode steps at position 2000, or two
    batched steps (what = the batch) at position 2000."""
    from . import cuda_abi, runtime
    dev = cuda_abi.Device(0)
    m = open_model(dev, name)
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
    a = ap.parse_args()
    once(a.size, a.what)
