"""Small models of listed layers for the tests: configurations, weights (BF16 values, so that BF16 and f32 models hold the
same numbers) and the comparison with the plain implementation in oracle/layered.py."""
import importlib
import os
import sys

import numpy as np

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

pkg = importlib.import_module("oxide-beta_b200")
syn = pkg.synthetic
from oracle import layered  # noqa: E402


def wkv(heads, dim, ff=None, **kw):
    return dict({"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": ff and {"kind": "dense", "ff": ff}}, **kw)


def lightning(heads, dim, vdim, decay, ff=None, **kw):
    return dict({"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)},
                 "mlp": ff and {"kind": "dense", "ff": ff}}, **kw)


def latent(heads, dim, vdim, q_rank, kv_rank, rot_dim, scale=None, base=10000.0, rot_dims=None, ff=None, **kw):
    return dict({"type": "latent_attention", "mlp": ff and {"kind": "dense", "ff": ff},
                 "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot_dim": rot_dim,
                           "rot": {"base": base, "dims": rot_dim if rot_dims is None else rot_dims},
                           "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}}, **kw)


def retention(heads, dim, vdim, decay, base=10000.0, rot_dims=None, ff=None, **kw):
    return dict({"type": "retention", "mlp": ff and {"kind": "dense", "ff": ff},
                 "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay),
                           "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims}}}, **kw)


def attention(heads, kv_heads, dim, vdim, scale=None, coef=0.7, every=5, ff=None, **kw):
    return dict({"type": "attention", "mlp": ff and {"kind": "dense", "ff": ff},
                 "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                           "scale": dim ** -0.5 if scale is None else scale, "q_temp": {"coef": coef, "every": every}}}, **kw)


def config(layers, width=100, vocab=333, eps=1e-5):
    parallel = layers[0]["type"] in ("retention", "attention")
    return {"architecture": "Nozurax" if parallel else "Pabovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


class Pair:
    """A device model and the plain implementation on the same weights."""

    def __init__(self, cfg, dtype="f32", seed=0, low_rank=11, edit=None):
        self.cfg, self.dtype = cfg, pkg.F32 if dtype == "f32" else pkg.BF16
        bits = dict(syn.layered_weights(cfg, seed, low_rank))
        if edit:
            for name, f in edit.items():
                bits[name] = syn.f32_to_bf16_bits(np.asarray(f(syn.bf16_bits_to_f32(bits[name])), dtype=np.float32))
        self.bits = bits
        self.W = {n: syn.bf16_bits_to_f32(a) for n, a in bits.items()}
        self.model = pkg.models.model_class(cfg).from_weights(cfg, bits, pkg.Device.Cuda(0), weight_dtype=self.dtype)
        self.state = self.model.prepare_cuda()

    def table(self, max_seq, batch=1, page_tokens=256, kv=None):
        return self.state.new_cache_table(max_seq, batch=batch, page_tokens=page_tokens, kv_dtype=self.dtype if kv is None else kv)

    def want(self, tokens):
        return layered.forward(self.cfg, self.W, tokens)[0]

    def prompt(self, n, seed=1):
        return syn.prompt_ids(self.cfg["vocab"], n, seed)


def error(got, want):
    """Largest over the rows of rms(difference, mean taken off) / rms of all wanted logits."""
    got, want = np.atleast_2d(np.asarray(got, np.float64)), np.atleast_2d(np.asarray(want, np.float64))
    d = got - want
    d -= d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt((w * w).mean()))


def feed(pair, table, tokens, portions):
    """Logits of every token, fed in portions of the given sizes (cycled); a portion of one is a decode step."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(portions[i % len(portions)], len(tokens) - at)
        if n == 1:
            out.append(pair.state.decode_token(int(tokens[at]), table)[None])
        else:
            out.append(pair.state.extend(tokens[at:at + n], table, want=range(n)))
        at += n
        i += 1
    return np.concatenate(out)
