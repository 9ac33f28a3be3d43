"""Nozurax models against the plain implementation of oracle/layered.py: every mechanism alone, prompts against token-by-token
decoding, portions, batches, reuse of cache tables, far keys, sinks, query temperature, first tokens, long decoding and
generation through the public entry point."""
import json
import os
import subprocess

import numpy as np
import pytest

from layered_util import ROOT, Pair, attention, config, error, feed, layered, pkg, retention, syn

pytestmark = pytest.mark.gpu

TOL = {"f32": 3e-5, "bf16": 3e-2}
# six random layers amplify a rounding (a head norm over an output close to zero most of all); a fault changes logits by their own size
DEEP = {"f32": 3e-5, "bf16": 0.2}
DTYPES = ("f32", "bf16")


def mixed():
    """Every mechanism in one odd-sized model: shared tensors, layers with and without feed-forward, one and several kv heads."""
    return config([attention(6, 2, 24, 20, ff=52), retention(3, 12, 28, (0.5, 0.93, 1.0), rot_dims=8, ff=50), attention(5, 1, 40, 56, every=1),
                   retention(2, 20, 12, (0.99, 0.7), base=300.0), attention(6, 2, 24, 20, ff=52, weights_of=0),
                   retention(3, 12, 28, (0.5, 0.93, 1.0), rot_dims=8, ff=50, weights_of=1)])


MECHANISMS = {
    "retention": [retention(3, 12, 28, (0.5, 0.93, 1.0))],
    "retention_partly_rotated": [retention(2, 40, 24, (0.9, 0.999), base=50.0, rot_dims=12)],
    "retention_not_rotated": [retention(2, 16, 16, (0.9, 0.99), rot_dims=0)],
    "retention_wide": [retention(2, 300, 40, (0.9, 0.999))],
    "retention_value_blocks": [retention(1, 48, 150, (0.97,), ff=40)],
    "retention_64": [retention(4, 64, 64, (0.9, 0.95, 0.99, 0.999), ff=64)],
    "retention_128": [retention(2, 128, 128, (0.97, 0.998))],
    "retention_odd": [retention(3, 10, 7, (0.6, 0.9, 0.99), rot_dims=6)],
    "attention": [attention(6, 2, 24, 20)],
    "attention_one_head": [attention(1, 1, 8, 8, ff=16)],
    "attention_own_kv": [attention(4, 4, 16, 48)],
    "attention_odd": [attention(3, 3, 9, 7, every=2)],
    "attention_20_heads_on_one": [attention(20, 1, 32, 16, coef=0.1, every=30)],
    "attention_100_by_128": [attention(4, 2, 100, 128)],
    "attention_200_by_256": [attention(4, 2, 200, 256)],
    "attention_256_by_40": [attention(2, 1, 256, 40)],
    "attention_too_wide_for_tensor_cores": [attention(3, 1, 300, 272)],
    "attention_cold": [attention(4, 2, 32, 32, scale=1.7, coef=0.0, every=7)],
    "attention_shared_tensors": [attention(4, 2, 16, 24, ff=32), retention(2, 12, 12, (0.9, 0.8)), attention(4, 2, 16, 24, ff=32, weights_of=0)],
    "feed_forward_odd": [retention(2, 8, 8, (0.5, 0.6), ff=37)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(name, dtype):
    """A whole prompt, then token by token from an empty table."""
    pair = Pair(config(MECHANISMS[name]), dtype, seed=3)
    tokens = pair.prompt(75)
    want = pair.want(tokens)
    assert error(feed(pair, pair.table(80), tokens, [75]), want) <= TOL[dtype]
    assert error(feed(pair, pair.table(80), tokens, [1]), want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 72, 97, 132])
def test_odd_widths(width, dtype):
    pair = Pair(config([attention(2, 1, 14, 18, ff=37), retention(2, 10, 11, (0.8, 0.95), ff=21)], width=width, vocab=131), dtype, seed=4)
    tokens = pair.prompt(40)
    want = pair.want(tokens)
    assert error(feed(pair, pair.table(40), tokens, [40]), want) <= TOL[dtype]
    assert error(feed(pair, pair.table(40), tokens, [1]), want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_eps_and_first_tokens(dtype):
    """A large eps, and requests of one, two and three tokens."""
    pair = Pair(config(mixed()["layers"], eps=0.3), dtype, seed=5)
    for n in (1, 2, 3):
        tokens = pair.prompt(n, seed=n)
        want = pair.want(tokens)
        for portions in ([n], [1], [2, 1]):
            assert error(feed(pair, pair.table(8), tokens, portions), want) <= DEEP[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", [[2], [3, 1, 2], [7, 37, 2, 2], [15, 16, 17], [31, 33], [64, 63, 65], [255, 2, 256], [400]])
def test_portions(portions, dtype):
    pair = Pair(mixed(), dtype, seed=6)
    tokens = pair.prompt(400)
    assert error(feed(pair, pair.table(400, page_tokens=48), tokens, portions), pair.want(tokens)) <= DEEP[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_logits_do_not_depend_on_pages_or_cache_type(dtype):
    pair = Pair(mixed(), dtype, seed=7)
    tokens = pair.prompt(130)
    want = pair.want(tokens)
    for page in (1, 7, 16, 256):
        assert error(feed(pair, pair.table(140, page_tokens=page), tokens, [100, 1]), want) <= DEEP[dtype]
    for kv in (pkg.F32, pkg.BF16):
        assert error(feed(pair, pair.table(140, kv=kv), tokens, [100, 1]), want) <= DEEP["bf16"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [2, 3, 9, 20])
def test_batch_of_unequal_requests_against_each_alone(batch, dtype):
    """Prompts of unequal length ingested together, then decoded together; some rows sit steps out."""
    pair = Pair(mixed(), dtype, seed=8)
    rng = np.random.default_rng(batch)
    lens = [int(n) for n in rng.integers(1, 90, size=batch)]
    lens[0] = 150
    tokens = [pair.prompt(n + 6, seed=20 + b) for b, n in enumerate(lens)]
    want = [pair.want(t) for t in tokens]
    table = pair.table([n + 8 for n in lens], batch=batch, page_tokens=32)
    got = pair.state.prefill_prompt(np.concatenate([t[:n] for t, n in zip(tokens, lens)]), table, lens=lens)
    for b in range(batch):
        assert error(got[b], want[b][lens[b] - 1]) <= DEEP[dtype], b
    done = [0] * batch
    for step in range(9):
        toks = np.full(batch, pkg.INACTIVE, dtype=np.uint32)
        for b in range(batch):
            if done[b] < 6 and (step + b) % 3 != 0:
                toks[b] = tokens[b][lens[b] + done[b]]
        got = pair.state.decode_token(toks, table)
        for b in range(batch):
            if toks[b] != pkg.INACTIVE:
                assert error(got[b], want[b][lens[b] + done[b]]) <= DEEP[dtype], (b, step)
                done[b] += 1
    assert [table.position(b) for b in range(batch)] == [n + d for n, d in zip(lens, done)]


@pytest.mark.parametrize("dtype", DTYPES)
def test_batch_portions_and_reused_sequences(dtype):
    """Portions of several sequences in one call, one sequence freed and used again while the others go on."""
    pair = Pair(mixed(), dtype, seed=9)
    tokens = [pair.prompt(n, seed=40 + i) for i, n in enumerate((120, 90, 61, 75))]
    want = [pair.want(t) for t in tokens]
    table = pair.table(128, batch=3, page_tokens=16)
    owner, at = [0, 1, 2], [0, 0, 0]
    for turn, lens in enumerate([(50, 2, 30), (0, 60, 31), (40, 28, 0), (2, 0, 50), (28, 0, 25)]):
        if turn == 3:                          # the third request is finished: its row serves the fourth one
            assert at[2] == 61
            table.reset_sequence(2)
            owner[2], at[2] = 3, 0
        flat = np.concatenate([tokens[owner[b]][at[b]:at[b] + lens[b]] for b in range(3)])
        got = pair.state.extend(flat, table, lens=list(lens), want=range(flat.size))
        i = 0
        for b in range(3):
            if lens[b]:
                assert error(got[i:i + lens[b]], want[owner[b]][at[b]:at[b] + lens[b]]) <= DEEP[dtype], (turn, b)
            i += lens[b]
            at[b] += lens[b]


@pytest.mark.parametrize("dtype", DTYPES)
def test_table_reuse_after_reset(dtype):
    pair = Pair(mixed(), dtype, seed=10)
    table = pair.table(100, page_tokens=16)
    for seed, n, portions in ((1, 100, [100]), (2, 40, [1]), (3, 70, [9, 1]), (4, 1, [1])):
        tokens = pair.prompt(n, seed=seed)
        assert error(feed(pair, table, tokens, portions), pair.want(tokens)) <= DEEP[dtype]
        table.reset()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens", [(65, 1, 64, 70, 2), (128, 66, 62), (64, 65, 127), (256, 3), (3, 253), (130, 126, 200)])
def test_runs_of_one_pass_of_all_lengths(lens, dtype):
    """Runs that are shorter than, as long as and longer than a block of the recurrence, side by side in one pass, then more of each."""
    pair = Pair(config([retention(2, 40, 36, (0.98, 0.9995)), retention(3, 10, 7, (0.9, 1.0, 0.5), rot_dims=6)]), dtype, seed=22)
    tokens = [pair.prompt(2 * n + 1, seed=60 + i) for i, n in enumerate(lens)]
    want = [pair.want(t) for t in tokens]
    table = pair.table([2 * n + 1 for n in lens], batch=len(lens))
    at = [0] * len(lens)
    for take in (lens, [n + 1 for n in lens]):
        flat = np.concatenate([t[a:a + n] for t, a, n in zip(tokens, at, take)])
        got = pair.state.extend(flat, table, lens=list(take), want=range(flat.size))
        i = 0
        for b, n in enumerate(take):
            assert error(got[i:i + n], want[b][at[b]:at[b] + n]) <= TOL[dtype], b
            i += n
            at[b] += n


def far_key_edits(dim):
    """Weights under which token 63 is the only one whose key answers to the query that all tokens share: channel 1 of the
    embedding feeds the query, channel 0, which only token 63 has, the key."""
    def embed(e):
        e = 0.5 * e
        e[:, 1] = 4.0
        e[:, 0] = 0.0
        e[63, 0] = 8.0
        return e

    def head_rows(col, value):
        def f(w):
            w = w.copy()
            w[::dim] = 0.0
            w[::dim, col] = value
            return w
        return f
    return {"embed": embed, "l0.mix.q": head_rows(1, 4.0), "l0.mix.k": head_rows(0, 9.0), "l0.mix.k.b": lambda b: 0.3 * b}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("key_at", [0, 1, 15, 16, 31, 32, 63, 64, 127, 128, 255, 256, 290])
def test_one_far_key_stands_out(key_at, dtype):
    """One key outweighs all others at every later position, however far back it is and wherever its page or tile ends."""
    cfg = config([attention(6, 2, 24, 32, scale=1.0, coef=0.3, every=50)], width=64, vocab=64)
    pair = Pair(cfg, dtype, seed=11, edit=far_key_edits(24))
    T = 300
    tokens = np.random.default_rng(key_at).integers(1, 63, size=T)
    without = tokens.copy()
    tokens[key_at] = 63
    want = pair.want(tokens)
    assert error(pair.want(without)[key_at + 1:], want[key_at + 1:]) > 0.4
    for page in (16, 64):
        assert error(feed(pair, pair.table(T, page_tokens=page), tokens, [280, 1]), want) <= TOL[dtype]
    assert error(feed(pair, pair.table(T), tokens, [key_at + 1, 5, 1, 2]), want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_sinks_take_their_share_once(dtype):
    """Sinks from nothing to nearly everything; the plain model without them, or counting them twice, is far off."""
    sinks = np.array([-8.0, 0.0, 3.0, 6.0, 9.0, 2.0])
    pair = Pair(config([attention(6, 3, 16, 16)], width=48, vocab=90), dtype, seed=19, edit={"l0.mix.sink": lambda s: sinks})
    tokens = pair.prompt(150)
    want = pair.want(tokens)
    for other in (sinks - 50.0, sinks + np.log(2.0)):
        assert error(layered.forward(pair.cfg, dict(pair.W, **{"l0.mix.sink": other}), tokens)[0], want) > 3 * TOL["bf16"]
    for portions in ([150], [1], [64, 1, 33]):
        assert error(feed(pair, pair.table(150), tokens, portions), want) <= TOL[dtype]
    both = pair.table(150, batch=2)
    got = pair.state.extend(np.concatenate([tokens, tokens[:70]]), both, lens=[150, 70], want=range(220))
    assert error(got, np.concatenate([want, want[:70]])) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("every", [1, 2, 16, 64])
def test_query_temperature_steps(every, dtype):
    """A strong temperature, so that a step one position early or late shows; prompts, portions and decoding around the steps."""
    pair = Pair(config([attention(4, 2, 32, 16, scale=0.2, coef=1.5, every=every)], width=48, vocab=90), dtype, seed=20)
    tokens = pair.prompt(140)
    want = pair.want(tokens)
    late = layered.query_temperature(np.arange(140) - 1, 1.5, every)
    now = layered.query_temperature(np.arange(140), 1.5, every)
    assert (late != now).sum() == (140 if every == 1 else 140 // every)
    for portions in ([140], [1], [15, 1, 2, 46]):
        assert error(feed(pair, pair.table(140), tokens, portions), want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_remember_the_first_token(dtype):
    """Decays close to one: the first token still shows hundreds of tokens later, and a lost or restarted state would too."""
    pair = Pair(config([retention(2, 16, 24, (1.0, 0.9995), base=1e6), retention(2, 16, 16, (0.999, 1.0))], width=48, vocab=100), dtype, seed=12)
    a = pair.prompt(500)
    b = a.copy()
    b[0] = (b[0] + 1) % 100
    want = pair.want(a)
    assert error(pair.want(b)[450:], want[450:]) > 3 * TOL["f32"]
    assert error(feed(pair, pair.table(500), a, [200, 1, 2, 37]), want) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_far_from_the_start(dtype):
    """Positions beyond 3000: angles of thousands of radians on the fast channels."""
    pair = Pair(config([retention(2, 16, 16, (0.99, 0.9), base=20.0)], width=32, vocab=60), dtype, seed=21)
    tokens = pair.prompt(3100)
    want = pair.want(tokens)
    got = feed(pair, pair.table(3200), tokens, [3080, 1])
    assert error(got[3000:], want[3000:]) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_and_fast_decay(dtype):
    """600 decode steps; decays from nothing to everything forgotten at once."""
    pair = Pair(config([retention(3, 8, 8, (1e-4, 0.99, 0.0)), attention(2, 1, 12, 20)], width=48, vocab=80), dtype, seed=13)
    tokens = pair.prompt(620)
    assert error(feed(pair, pair.table(620), tokens, [20] + [1] * 600), pair.want(tokens)) <= TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_layer_trace(dtype):
    """The residual stream at every layer of decode steps."""
    pair = Pair(mixed(), dtype, seed=14)
    tokens = pair.prompt(12)
    _, after = layered.forward(pair.cfg, pair.W, tokens)
    table = pair.table(16)
    for t, tok in enumerate(tokens):
        trace, logits = pair.state.decode_trace(int(tok), table)
        assert error(trace[1:, 0], after[:, t]) <= DEEP[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_public_entry_point(dtype, tmp_path):
    """config.json + model.safetensors through the registry, generate(), the device loop and the batch path."""
    cfg = mixed()
    pair = Pair(cfg, dtype, seed=15)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    syn.write_tensors(str(tmp_path / "model.safetensors"), pair.bits.items())
    model = pkg.load_pretrained(str(tmp_path), pkg.Device.Cuda(0), weight_dtype=pair.dtype)
    assert type(model) is pkg.NozuraxForCausalLM
    prompt = [int(t) for t in pair.prompt(30)]
    out = model.generate(prompt, pkg.GenerationConfig.greedy(24))
    assert out[:30] == prompt and len(out) == 54
    logits = pair.want(out[:-1])[29:]
    for i, tok in enumerate(out[30:]):            # every choice is the plain implementation's, or within rounding of it
        assert logits[i].max() - logits[i][tok] <= DEEP[dtype] * np.abs(logits[i]).max()
    streamed = []
    assert model.generate_stream(prompt, pkg.GenerationConfig.greedy(24), streamed.append) == out and streamed == out[30:]
    table = pair.table(64)
    first = int(np.argmax(pair.state.prefill_prompt(prompt, table)))
    ids, _ = pair.state.decode_greedy([first], table, 23)
    assert [first] + [int(i) for i in ids[:, 0]] == out[30:]
    both = pair.table(64, batch=2)
    pair.state.prefill_prompt(prompt + prompt[:9], both, lens=[30, 9])
    ids, _ = pair.state.decode_greedy([first, 5], both, 23)
    if dtype == "f32":
        assert [first] + [int(i) for i in ids[:, 0]] == out[30:]
    sampled = model.generate(prompt, pkg.GenerationConfig(max_new_tokens=10, top_k=8, eos_token_ids=[]))
    assert len(sampled) == 40 and max(sampled) < cfg["vocab"]


def test_graph_replay_equals_eager_launches(monkeypatch):
    pair = Pair(mixed(), "bf16", seed=16)
    tokens = pair.prompt(40)
    a = feed(pair, pair.table(40), tokens, [20, 1])
    monkeypatch.setenv("GEMMA4_DISABLE_CUDA_GRAPH", "1")
    b = feed(pair, pair.table(40), tokens, [20, 1])
    assert np.array_equal(a, b)


def test_profiles():
    pair = Pair(mixed(), "bf16", seed=17)
    table = pair.table(64)
    prof = pair.state.profile_extend(pair.prompt(20), table)
    assert {"qkv", "recur", "qkv_post", "attn", "attn_merge", "outnorm", "o"} <= set(prof) and table.position() == 20
    assert "gateup" not in prof and "down" not in prof
    assert {"qkv", "recur", "attn", "o"} <= set(pair.state.profile_step([1], table))


def test_trace_replay(tmp_path):
    """bin/trace_run: two requests one after the other, the second in the table the first gave back."""
    pair = Pair(mixed(), "bf16", seed=18)
    (tmp_path / "config.json").write_text(json.dumps(pair.cfg))
    syn.write_tensors(str(tmp_path / "model.safetensors"), pair.bits.items())
    a, b = pair.prompt(33, seed=1), pair.prompt(21, seed=2)
    steps = [("a", a[:30], [3, 29], []), ("a", a[30:31], [0], []), ("a", a[31:], [1], ["a"]), ("b", b[:20], [], []), ("b", b[20:], [0], ["b"])]
    lines = "".join(json.dumps({"step": n, "entries": [{"id": i, "tokens": [int(t) for t in tok], "want": w}], "end": end}) + "\n"
                    for n, (i, tok, w, end) in enumerate(steps))
    want = {"a": pair.want(a), "b": pair.want(b)}
    for dtype in ("bfloat16", "float32"):
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                              "--max-tokens", "40"], input=lines, capture_output=True, text=True, timeout=300)
        assert run.returncode == 0, run.stderr[-2000:]
        assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {n}" for n in range(5)]
        at = {"a": 0, "b": 0}
        for n, (i, tok, w, _) in enumerate(steps):
            f = tmp_path / f"{n}.f32"
            if w:
                got = np.fromfile(f, dtype="<f4").reshape(len(w), -1)
                assert error(got, want[i][[at[i] + p for p in w]]) <= DEEP["bf16" if dtype == "bfloat16" else "f32"]
                f.unlink()
            at[i] += len(tok)
