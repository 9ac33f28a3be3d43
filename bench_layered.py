"""Throughput of models of listed layers beside models of equal width, depth, feed-forward and vocabulary: Gemma 4, and for
Nozurax (whose recurrence is like lightning attention) also Pabovik. Run through `python bench.py --design pabovik|nozurax`;
prints ONE JSON line.

Per size and model: prefill tokens/s (one prompt of 4096 tokens in one call, host clock around the call, which ends with a
synchronisation), decode tokens/s of the captured greedy step (CUDA events on the library's stream) for one sequence and for
a batch of 32 behind contexts of 4096, and the device time of every kernel kind per launch from eager profiling passes,
with the bytes or FLOPs it has to move and the fraction of the roofline that is. Weights are random; weights and caches
exceed L2.
"""
import importlib
import json
import os
import sys
import time

import numpy as np

ROOT = os.path.dirname(os.path.abspath(__file__))
CONTEXT, BATCH = 4096, 32


def peaks():
    p = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(p):
        with open(p) as f:
            d = json.load(f)
        return float(d["hbm_gbs"]) * 1e9, float(d["bf16_tflops"]) * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def sizes(design):
    """name -> {model: config} of equal width, depth, feed-forward and vocabulary, the design's own first."""
    syn = importlib.import_module("oxide-beta_b200").synthetic
    out = {}
    for name, width, heads, ff, q_rank in (("w2560", 2560, 16, 10240, 1024), ("w4096", 4096, 32, 14336, 1536)):
        wkv = {"type": "wkv", "mixer": {"heads": width // 64, "dim": 64}, "mlp": {"kind": "dense", "ff": ff}}
        lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff},
               "mixer": {"heads": heads, "dim": 128, "vdim": 128, "q_rank": q_rank, "kv_rank": 512, "rot_dim": 64,
                         "rot": {"dims": 64, "base": 10000.0}, "scale": 192 ** -0.5}}
        lit = {"type": "lightning", "mlp": {"kind": "dense", "ff": ff},
               "mixer": {"heads": width // 128, "dim": 128, "vdim": 128,
                         "decay": [float(np.exp(-2.0 ** (-8.0 * (h + 1) / (width // 128)))) for h in range(width // 128)]}}
        layers = [wkv, lat, lit] * 4
        models = {"pabovik": {"architecture": "Pabovik", "vocab": 65536, "width": width, "norm": {"eps": 1e-6}, "layers": layers},
                  "gemma4": syn._cfg(65536, width, len(layers), heads // 2, heads // 4, 256, ff, 1024)}
        if design == "nozurax":
            att = {"type": "attention", "mlp": {"kind": "dense", "ff": ff},
                   "mixer": {"heads": width // 128, "kv_heads": width // 512, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                             "q_temp": {"coef": 0.1, "every": 8192}}}
            ret = {"type": "retention", "mlp": {"kind": "dense", "ff": ff},
                   "mixer": dict(lit["mixer"], rot={"dims": 128, "base": 10000.0})}
            models = {"nozurax": {"architecture": "Nozurax", "vocab": 65536, "width": width, "norm": {"eps": 1e-6},
                                  "layers": [att, ret] * (len(layers) // 2)}, **models}
        out[name] = models
    return out


def device_weights(names):
    """Random BF16 bit patterns drawn on the GPU, tensor by tensor."""
    import torch
    gen = torch.Generator(device="cuda").manual_seed(0)
    for name, shape, kind in names:
        t = torch.empty(shape, dtype=torch.float32, device="cuda")
        if kind in ("matrix",):
            t.normal_(0.0, shape[-1] ** -0.5, generator=gen)
        elif kind in ("norm0", "bias", "sink"):
            t.normal_(0.0, 0.2, generator=gen)
        elif kind == "w0":
            t.uniform_(-6.0, 0.5, generator=gen)
        elif kind == "mu":
            t.uniform_(0.0, 1.0, generator=gen)
        else:
            t.fill_(1.0)
        yield name, t.to(torch.bfloat16).view(torch.int16).cpu().numpy().view(np.uint16)


def work(cfg, kind, rows, contexts, chunk):
    """(bytes, flops) one launch of a kernel kind has to move / do, averaged over the layers that launch it; a chunk's rows
    attend to `contexts` positions on average."""
    got = []
    for layer in cfg["layers"]:
        c, H, t = layer["mixer"], cfg["width"], layer["type"]
        ff = layer["mlp"]["ff"]
        heads, dim = c["heads"], c["dim"]
        vdim = c.get("vdim", dim)

        def gemm(n, k, heads_=1):
            return heads_ * (2 * n * k + 2 * rows * k + 4 * rows * n), heads_ * 2 * n * k * rows

        if t in ("attention", "retention"):
            # mixer, gate and up rows are one input projection, mixer and feed-forward columns one output projection
            kvh = c.get("kv_heads")
            if kind == "o":
                got.append(gemm(H, heads * vdim + ff))
            elif kind == "qkv":
                got.append(gemm(2 * ff + (heads * dim + kvh * (dim + vdim) if kvh else 2 * heads * (dim + vdim)), H))
            elif kvh and kind == "attn":
                seqs = 1 if chunk else rows
                got.append((2 * seqs * contexts * kvh * (dim + vdim), 2 * rows * heads * contexts * (dim + vdim)))
            elif not kvh and kind == "recur":
                got.append((8 * (1 if chunk else rows) * heads * dim * vdim + 4 * rows * heads * 2 * (dim + vdim),
                            6 * rows * heads * dim * vdim))
        elif kind == "gateup":
            got.append(gemm(2 * ff, H))
        elif kind == "down":
            got.append(gemm(H, ff))
        elif kind == "o":
            got.append(gemm(H, heads * vdim))
        elif kind == "qkv":
            n = (4 * heads * dim + 64 if t == "wkv" else 2 * heads * (dim + vdim) if t == "lightning" else
                 c["q_rank"] + c["kv_rank"] + c["rot_dim"] + heads * vdim)
            got.append(gemm(n, H))
        elif t == "latent_attention" and kind == "uq":
            got.append(gemm(heads * (dim + c["rot_dim"]), c["q_rank"]))
        elif t == "latent_attention" and kind in ("uk", "latq"):
            got.append(gemm(c["kv_rank"], dim, heads))
        elif t == "latent_attention" and kind in ("uv", "latout"):
            got.append(gemm(vdim, c["kv_rank"], heads))
        elif t == "latent_attention" and kind == "attn":
            seqs = 1 if chunk else rows
            ld = c["kv_rank"] + c["rot_dim"]
            got.append((2 * seqs * contexts * ld, 2 * rows * heads * contexts * (ld + c["kv_rank"])))
        elif t != "latent_attention" and kind == "recur":
            seqs = 1 if chunk else rows
            streams = (5 if t == "wkv" else 4) * heads * dim
            got.append((8 * seqs * heads * dim * vdim + 4 * rows * streams, 6 * rows * heads * dim * vdim))
    return tuple(float(np.mean(x)) for x in zip(*got)) if got else None


def gemma_work(cfg, kind, rows, contexts, chunk):
    H, I, D = cfg["hidden_size"], cfg["intermediate_size"], cfg["head_dim"]
    Nq, Nkv = cfg["num_attention_heads"], cfg["num_key_value_heads"]

    def gemm(n, k):
        return 2 * n * k + 2 * rows * k + 4 * rows * n, 2 * n * k * rows

    if kind == "attn":
        vis = np.mean([contexts if t == "full_attention" else min(contexts, cfg["sliding_window"]) for t in cfg["layer_types"]])
        seqs = 1 if chunk else rows
        return 4 * seqs * vis * Nkv * D, 4 * rows * Nq * vis * D
    return {"gateup": gemm(2 * I, H), "down": gemm(H, I), "o": gemm(H, Nq * D), "qkv": gemm((Nq + 2 * Nkv) * D, H)}.get(kind)


def kernel_table(prof, counter, rows, contexts, chunk):
    hbm, tf, _ = peaks()
    out = {}
    for kind, ms in sorted(prof.items(), key=lambda x: -x[1]):
        w = counter(kind, rows, contexts, chunk)
        row = {"us": round(1000 * ms, 2)}
        if w:
            # the recurrences run on the f32 pipes (128 lanes x 148 SMs x 2 at 1.9 GHz), everything else on the tensor cores
            peak = 128 * 148 * 2 * 1.9e9 if kind == "recur" else tf
            need = max(w[0] / hbm, w[1] / peak)
            row.update(bound="hbm" if w[0] / hbm >= w[1] / peak else "flops", roofline_frac=round(need / (ms * 1e-3), 3))
        out[kind] = row
    return out


def measure(pkg, state, vocab, counter):
    syn = pkg.synthetic
    res = {}
    prompt = syn.prompt_ids(vocab, CONTEXT, seed=1)
    table = state.new_cache_table(CONTEXT + 600, kv_dtype=pkg.BF16)
    state.prefill_prompt(prompt, table)                                   # warm-up
    best = 1e9
    for _ in range(3):
        table.reset()
        t0 = time.perf_counter()
        logits = state.prefill_prompt(prompt, table)
        best = min(best, time.perf_counter() - t0)
    res["prefill_tok_s"] = round(CONTEXT / best, 1)
    table.reset()
    state.extend(prompt[:CONTEXT - 256], table)
    res["prefill_kernels"] = kernel_table(state.profile_extend(prompt[-256:], table), counter, 256, CONTEXT - 128, True)
    res["prefill_chunk_us"] = {k: round(1000 * v, 1) for k, v in _totals(state).items()}
    first = [int(np.argmax(logits))]
    ids, _ = state.decode_greedy(first, table, 32)
    ids, ms = state.decode_greedy(ids[-1], table, 128)
    res["decode_b1_tok_s"], res["decode_b1_ms"] = round(1000.0 / ms, 1), round(ms, 4)
    state.profile_step(ids[-1], table)
    res["decode_b1_kernels"] = kernel_table(state.profile_step(ids[-1], table), counter, 1, CONTEXT + 160, False)
    res["decode_b1_us"] = {k: round(1000 * v, 1) for k, v in _totals(state).items()}
    table.close()
    table = state.new_cache_table([CONTEXT + 300] * BATCH, batch=BATCH, kv_dtype=pkg.BF16)
    table.fill_synthetic([CONTEXT] * BATCH)
    ids, _ = state.decode_greedy(np.arange(BATCH) * 7 % vocab, table, 16)
    ids, ms = state.decode_greedy(ids[-1], table, 64)
    res[f"decode_b{BATCH}_tok_s"], res[f"decode_b{BATCH}_ms"] = round(1000.0 * BATCH / ms, 1), round(ms, 4)
    state.profile_step(ids[-1], table)
    res[f"decode_b{BATCH}_kernels"] = kernel_table(state.profile_step(ids[-1], table), counter, BATCH, CONTEXT + 80, False)
    res[f"decode_b{BATCH}_us"] = {k: round(1000 * v, 1) for k, v in _totals(state).items()}
    table.close()
    return res


def _totals(state):
    return state._profile(True)


def main(design):
    import torch
    if not torch.cuda.is_available():
        raise SystemExit("the benchmark needs a CUDA device: the library has no CPU path")
    sys.stdout.flush()
    json_fd = os.dup(1)
    os.dup2(2, 1)
    pkg = importlib.import_module("oxide-beta_b200")
    syn = pkg.synthetic
    hbm, tf, kind = peaks()
    out = {"design": design, "data": "synthetic", "dtype": "bf16", "context": CONTEXT, "batch": BATCH,
           "peaks": {"hbm_gbs": hbm / 1e9, "bf16_tflops": tf / 1e12, "kind": kind}, "sizes": {}}
    for name, models in sizes(design).items():
        r = {}
        for model, cfg in models.items():
            if model == "gemma4":
                state, counter = pkg.Gemma4CudaState.load(pkg.Gemma4TextConfig(cfg), device_weights(syn.weight_names(cfg))), gemma_work
            else:
                cls = pkg.models.model_class(cfg)
                state = cls.STATE.load(cls.CONFIG(cfg), device_weights(syn.layered_weight_names(cfg, low_rank=64)))
                counter = work
            r[model] = {"weight_gb": round(state.weight_bytes() / 1e9, 3),
                        **measure(pkg, state, state.config.vocab_size, lambda k, n, c, ch: counter(cfg, k, n, c, ch))}
            state.close()
        out["sizes"][name] = r
    sys.stdout.flush()
    os.write(json_fd, (json.dumps(out) + "\n").encode())
