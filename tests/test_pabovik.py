"""CPU tests of models of listed layers: configuration, registry, checkpoint files, the native boundary, and the plain
implementation itself."""
import json
import os
import re

import numpy as np
import pytest

from layered_util import ROOT, config, layered, lightning, latent, pkg, syn, wkv

N = pkg._native


def small():
    return config([wkv(2, 12, ff=20), latent(3, 8, 10, 16, 24, 6), lightning(2, 8, 14, (0.5, 0.9)), lightning(2, 8, 14, (0.5, 0.9), weights_of=2)], width=40, vocab=50)


def test_struct_layouts_match_header():
    header = open(os.path.join(ROOT, "include", "oxg4.h")).read()
    for struct, cls in (("oxg4_layer_spec", N.LayerSpec), ("oxg4_layered_config", N.LayeredConfig)):
        body = re.search(r"typedef struct \{([^}]*)\} %s;" % struct, header, re.S).group(1)
        names = re.findall(r"(\w+);", re.sub(r"/\*.*?\*/", "", body, flags=re.S))
        assert names == [f[0] for f in cls._fields_]


def test_registry_and_checkpoint(tmp_path):
    cfg = small()
    bits = dict(syn.layered_weights(cfg, 1, low_rank=5))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    syn.write_tensors(str(tmp_path / "model.safetensors"), bits.items())
    m = pkg.load_pretrained(str(tmp_path), pkg.Device.Cpu())
    assert type(m) is pkg.PabovikForCausalLM and m.config().num_hidden_layers == 4
    assert np.array_equal(m.weight("l0.mix.w1"), bits["l0.mix.w1"])
    assert m.embed([3, 7]).shape == (2, 40)
    with pytest.raises(pkg.Oxg4Error, match="Device::Cuda"):
        m.generate([1], pkg.GenerationConfig.greedy(1))
    assert pkg.models.model_class({"model_type": "gemma4"}) is pkg.Gemma4ForCausalLM
    with pytest.raises(pkg.Oxg4Error, match="no model"):
        pkg.models.model_class({"architecture": "other"})


def test_configuration_is_read_and_checked():
    cfg = pkg.PabovikConfig(small())
    native, keep = cfg.native(pkg.BF16)
    s = native.layers
    assert (s[0].mixer, s[0].heads, s[0].dim, s[0].vdim, s[0].ff, s[0].weights_of) == (3, 2, 12, 12, 20, -1)
    assert (s[1].q_rank, s[1].kv_rank, s[1].rot_dim, s[1].rot_dims, s[1].ff) == (16, 24, 6, 6, 0)
    assert s[3].weights_of == 2 and s[2].decay[1] == np.float32(0.9)
    for edit, msg in ((lambda c: c["layers"][0].update(type="rnn"), "unknown mixer"),
                      (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
                      (lambda c: c.pop("width"), "invalid Pabovik configuration")):
        bad = small()
        edit(bad)
        with pytest.raises(pkg.Oxg4Error, match=msg):
            pkg.PabovikConfig(bad)
    bad = small()
    bad["layers"][2]["mixer"]["decay"] = [0.5]
    with pytest.raises(pkg.Oxg4Error, match="one decay per head"):
        pkg.PabovikConfig(bad).native(pkg.BF16)
    bad = small()
    bad["layers"][2]["weights_of"] = 3
    with pytest.raises(pkg.Oxg4Error, match="weights_of"):
        pkg.PabovikConfig(bad).native(pkg.BF16)


def test_checkpoint_with_missing_or_misshapen_tensors_is_refused():
    bits = dict(syn.layered_weights(small(), 1, low_rank=5))
    short = dict(bits)
    del short["l1.mix.uk"]
    with pytest.raises(pkg.Oxg4Error, match="missing `l1.mix.uk`"):
        pkg.PabovikForCausalLM.from_weights(small(), short, pkg.Device.Cpu())
    with pytest.raises(pkg.Oxg4Error, match="l0.mix.w2"):
        pkg.PabovikForCausalLM.from_weights(small(), dict(bits, **{"l0.mix.w2": bits["l0.mix.w2"][:, :4]}), pkg.Device.Cpu())


def test_library_checks_sizes_before_it_looks_for_a_device():
    bad = small()
    bad["layers"][1]["mixer"]["rot"]["dims"] = 8
    with pytest.raises(pkg.Oxg4Error, match="latent attention sizes"):
        pkg.PabovikCudaState(pkg.PabovikConfig(bad))
    bad = small()
    bad["layers"][1]["mixer"]["kv_rank"] = 600
    with pytest.raises(pkg.Oxg4Error, match="kv_rank above 512"):
        pkg.PabovikCudaState(pkg.PabovikConfig(bad))
    import torch
    if not torch.cuda.is_available():
        with pytest.raises(pkg.Oxg4Error, match="no CPU path"):
            pkg.PabovikCudaState(pkg.PabovikConfig(small()))


def test_plain_mechanisms_against_their_closed_forms():
    rng = np.random.default_rng(0)
    T, H, D, Dv = 9, 2, 4, 3
    q, k = rng.standard_normal((2, T, H, D))
    v = rng.standard_normal((T, H, Dv))
    decay = np.array([0.5, 1.0])
    got = layered.lightning_scan(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            o = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            np.testing.assert_allclose(got[t, h], o, rtol=1e-10)
    w, u = rng.uniform(0.1, 1.0, (T, H, D)), rng.standard_normal((H, D))
    vv = rng.standard_normal((T, H, D))
    got = layered.wkv_scan(q, k, vv, w, u)
    for t in range(T):
        for h in range(H):
            o = (q[t, h] * u[h]) @ k[t, h] * vv[t, h]
            for s in range(t):
                o = o + (q[t, h] * np.prod(w[s + 1:t, h], axis=0)) @ k[s, h] * vv[s, h]
            np.testing.assert_allclose(got[t, h], o, rtol=1e-9)
    # turning queries and keys alike leaves their product a function of the distance
    x, y = rng.standard_normal((2, 1, 1, 8))
    dots = [float((layered.rotate_interleaved(x, [p + 5], 8, 100.0) * layered.rotate_interleaved(y, [p], 8, 100.0)).sum()) for p in (0, 3, 90)]
    np.testing.assert_allclose(dots, dots[0], rtol=1e-9)
    h = rng.standard_normal((3, 5))
    np.testing.assert_allclose(layered.token_shift_mix(h, np.full(5, 1.0))[1:], h[:-1])
    assert not layered.token_shift_mix(h, np.full(5, 1.0))[0].any()


def test_plain_model_is_causal_and_shares_tensors():
    cfg = small()
    W = {n: syn.bf16_bits_to_f32(a) for n, a in syn.layered_weights(cfg, 1, low_rank=5)}
    tokens = syn.prompt_ids(50, 20, 3)
    logits, after = layered.forward(cfg, W, tokens)
    assert after.shape == (4, 20, 40)
    np.testing.assert_allclose(layered.forward(cfg, W, tokens[:11])[0], logits[:11], rtol=1e-9, atol=1e-12)
    own = json.loads(json.dumps(cfg))
    del own["layers"][3]["weights_of"]
    W2 = dict(W, **{n.replace("l2.", "l3."): a for n, a in W.items() if n.startswith("l2.")})
    np.testing.assert_allclose(layered.forward(own, W2, tokens)[0], logits)
