"""CPU tests of Nozurax models: configuration, registry, checkpoint files, the native boundary, and the plain implementation
itself."""
import json

import numpy as np
import pytest

from layered_util import attention, config, latent, layered, pkg, retention, syn

N = pkg._native


def small():
    return config([attention(6, 2, 8, 10, scale=0.3, coef=0.5, every=4, ff=20), retention(2, 12, 14, (0.5, 0.9), base=700.0, rot_dims=6),
                   retention(2, 12, 14, (0.5, 0.9), base=700.0, rot_dims=6, weights_of=1)], width=40, vocab=50)


def test_registry_and_checkpoint(tmp_path):
    cfg = small()
    bits = dict(syn.layered_weights(cfg, 1))
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    syn.write_tensors(str(tmp_path / "model.safetensors"), bits.items())
    m = pkg.load_pretrained(str(tmp_path), pkg.Device.Cpu())
    assert type(m) is pkg.NozuraxForCausalLM and isinstance(m, pkg.LayeredForCausalLM) and m.config().num_hidden_layers == 3
    assert np.array_equal(m.weight("l0.mix.sink"), bits["l0.mix.sink"]) and not any(n.startswith("l2.") for n in bits)
    assert m.embed([3, 7]).shape == (2, 40)
    with pytest.raises(pkg.Oxg4Error, match="Device::Cuda"):
        m.generate([1], pkg.GenerationConfig.greedy(1))
    with pytest.raises(pkg.Oxg4Error, match="Nozurax generate requires Device::Cuda"):
        m.prepare_cuda()
    for name, change in (("l0.mix.q.b", lambda a: a[:-1]), ("l1.mix.g", lambda a: a[:, :-1]), ("final.norm", lambda a: a[1:])):
        with pytest.raises(pkg.Oxg4Error, match=name):
            pkg.NozuraxForCausalLM.from_weights(cfg, dict(bits, **{name: change(bits[name])}), pkg.Device.Cpu())
    del bits["l0.mix.sink"]
    with pytest.raises(pkg.Oxg4Error, match="missing `l0.mix.sink`"):
        pkg.NozuraxForCausalLM.from_weights(cfg, bits, pkg.Device.Cpu())


def test_configuration_is_read_and_checked():
    native, keep = pkg.NozuraxConfig(small()).native(pkg.BF16)
    s = native.layers
    assert (native.block, native.act, native.norm_weight_offset) == (N.BLOCK_PARALLEL, N.ACTIVATIONS["relu"], 1)
    assert (s[0].mixer, s[0].heads, s[0].kv_heads, s[0].dim, s[0].vdim, s[0].ff, s[0].q_temp_every) == (5, 6, 2, 8, 10, 20, 4)
    assert s[0].q_temp_coef == 0.5 and s[0].scale == np.float32(0.3)
    assert (s[1].mixer, s[1].dim, s[1].vdim, s[1].rot_dims, s[1].rot_base, s[1].ff) == (4, 12, 14, 6, 700.0, 0)
    assert s[1].decay[1] == np.float32(0.9) and (s[1].weights_of, s[2].weights_of) == (-1, 1)
    assert pkg.PabovikConfig({"vocab": 9, "width": 8, "norm": {"eps": 1e-5}, "layers": []}).native(pkg.F32)[0].block == N.BLOCK_SANDWICH
    for edit, msg in ((lambda c: c["layers"][0].update(type="latent_attention"), "unknown mixer"),
                      (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "unknown feed-forward"),
                      (lambda c: c.pop("norm"), "invalid Nozurax configuration"),
                      (lambda c: c["layers"][0]["mixer"].pop("q_temp"), "invalid Nozurax configuration"),
                      (lambda c: c["layers"][1]["mixer"].pop("decay"), "invalid Nozurax configuration"),
                      (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "one decay per head"),
                      (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=2.5), "whole number"),
                      (lambda c: c["layers"][2].update(weights_of=2), "weights_of")):
        bad = small()
        edit(bad)
        with pytest.raises(pkg.Oxg4Error, match=msg):
            pkg.NozuraxConfig(bad).native(pkg.BF16)


def test_library_checks_sizes_before_it_looks_for_a_device():
    for edit, msg in ((lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple of kv heads"),
                      (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "q_temp_every"),
                      (lambda c: c["layers"][0]["mixer"].update(vdim=600), "value size above 512"),
                      (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=14), "invalid rotation"),
                      (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5), "invalid rotation"),
                      (lambda c: c["layers"][1]["mixer"].update(dim=600), "key size above 512")):
        bad = small()
        edit(bad)
        with pytest.raises(pkg.Oxg4Error, match=msg):
            pkg.NozuraxCudaState(pkg.NozuraxConfig(bad))

    class Mixed(pkg.NozuraxConfig):
        MIXERS = ("retention", "latent_attention")

        def mixer_spec(self, layer, s):
            (pkg.PabovikConfig if layer["type"] == "latent_attention" else pkg.NozuraxConfig).mixer_spec(self, layer, s)
    with pytest.raises(pkg.Oxg4Error, match="not available in block"):
        pkg.NozuraxCudaState(Mixed(config([retention(1, 8, 8, (0.5,)), latent(1, 8, 8, 8, 8, 4)], width=16, vocab=20)))


def test_plain_mechanisms_against_their_closed_forms():
    rng = np.random.default_rng(0)
    # turning queries and keys alike leaves their product a function of the distance; the rest of a head does not turn
    x, y = rng.standard_normal((2, 1, 1, 10))
    dots = [float((layered.rotate_half(x, [p + 5], 8, 100.0) * layered.rotate_half(y, [p], 8, 100.0)).sum()) for p in (0, 3, 90)]
    np.testing.assert_allclose(dots, dots[0], rtol=1e-9)
    turned = layered.rotate_half(x, [7], 8, 100.0)
    np.testing.assert_array_equal(turned[..., 8:], x[..., 8:])
    c, s = np.cos(7 * 100.0 ** -0.25), np.sin(7 * 100.0 ** -0.25)
    np.testing.assert_allclose(turned[0, 0, [1, 5]], [x[0, 0, 1] * c - x[0, 0, 5] * s, x[0, 0, 5] * c + x[0, 0, 1] * s])
    # a sink is one more key of that score whose value is zero
    q, k = rng.standard_normal((2, 6, 2, 4))
    v, sink = rng.standard_normal((6, 2, 3)), np.array([0.7, -2.0])
    got = layered.causal_softmax_attention(q, k, v, 0.5, sink)
    for t in range(6):
        for h in range(2):
            e = np.exp(np.append(0.5 * k[:t + 1, h] @ q[t, h], sink[h]))
            np.testing.assert_allclose(got[t, h], (e[:-1] / e.sum()) @ v[:t + 1, h], rtol=1e-10)
    np.testing.assert_allclose(layered.query_temperature([0, 2, 3, 6, 7], 0.5, 4), 1 + 0.5 * np.log([1, 1, 2, 2, 3]))


def test_plain_model_is_causal_and_shares_tensors():
    cfg = small()
    W = {n: syn.bf16_bits_to_f32(a) for n, a in syn.layered_weights(cfg, 1)}
    tokens = syn.prompt_ids(50, 20, 3)
    logits, after = layered.forward(cfg, W, tokens)
    assert after.shape == (3, 20, 40)
    np.testing.assert_allclose(layered.forward(cfg, W, tokens[:11])[0], logits[:11], rtol=1e-9, atol=1e-12)
    own = json.loads(json.dumps(cfg))
    del own["layers"][2]["weights_of"]
    W2 = dict(W, **{n.replace("l1.", "l2."): a for n, a in W.items() if n.startswith("l1.")})
    np.testing.assert_allclose(layered.forward(own, W2, tokens)[0], logits)


def test_mixer_and_feed_forward_read_the_same_input():
    """x + mixer(h) + ff(h) with h = norm(x): each part alone, and the norm's weight around zero."""
    cfg = config([retention(2, 12, 14, (0.5, 0.9), ff=24)], width=40, vocab=50)
    W = {n: np.asarray(syn.bf16_bits_to_f32(a), np.float64) for n, a in syn.layered_weights(cfg, 2)}
    tokens = syn.prompt_ids(50, 12, 3)
    x = W["embed"][tokens]
    h = x / np.sqrt((x * x).mean(-1, keepdims=True) + 1e-5) * (1 + W["l0.norm1"])
    mix = layered.retention(h, W, "l0.", cfg["layers"][0]["mixer"], 1e-5)
    ff = (np.maximum(h @ W["l0.mlp.gate"].T, 0) * (h @ W["l0.mlp.up"].T)) @ W["l0.mlp.down"].T
    np.testing.assert_allclose(layered.forward(cfg, W, tokens)[1][0], x + mix + ff, rtol=1e-10)
