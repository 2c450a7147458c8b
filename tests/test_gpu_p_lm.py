"""Decoder language models on the GPU against the plain statement of the design (lm_plain.py), through
the library's own step function, slots and generation loop."""
import json
import os
import subprocess

import numpy as np
import pytest

import lm_plain as plain
from lm_models import DTYPES, LIMIT, Case, attention, config, delta, error, feed, tokens, weights, write_folder

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def lm_mod(pkg):
    return pkg


MECHANISMS = {
    # gated delta rule
    "delta": [delta()],
    "delta_equal_heads": [delta(heads=2, kv_heads=2, dim=16, vdim=16, conv=4)],
    "delta_no_taps": [delta(conv=1)],
    "delta_many_taps": [delta(conv=6, heads=6, kv_heads=3, dim=20, vdim=36)],
    "delta_odd_sizes": [delta(heads=5, kv_heads=1, dim=37, vdim=51, ff=0)],
    "delta_large_heads": [delta(heads=2, kv_heads=1, dim=128, vdim=160, conv=2, ff=0)],
    "delta_wide_keys": [delta(heads=2, kv_heads=2, dim=200, vdim=64, ff=0)],
    # attention
    "attention": [attention()],
    "attention_causal": [attention(window=0)],
    "attention_keep_none": [attention(keep=0)],
    "attention_window_one": [attention(window=1, keep=2)],
    "attention_keep_past_window": [attention(window=4, keep=40)],
    "attention_no_softcap": [attention(softcap=0)],
    "attention_low_softcap": [attention(softcap=1.5)],
    "attention_plain_rope": [attention(scaling=None)],
    "attention_no_rope": [attention(rot=0)],
    "attention_full_rope": [attention(rot=32, base=300.0, scaling={"factor": 8.0, "original": 90, "fast": 4.0, "slow": 1.0})],
    "attention_rope_two": [attention(rot=2)],
    "attention_sizes": [attention(heads=9, kv_heads=3, dim=20, vdim=12, rot=10, ff=0)],
    "attention_odd_sizes": [attention(heads=3, kv_heads=1, dim=27, vdim=33, rot=6, ff=0)],
    "attention_one_kv": [attention(heads=20, kv_heads=1, dim=16, vdim=24, rot=8)],
    "attention_mha": [attention(heads=3, kv_heads=3, dim=64, vdim=64, rot=64)],
    "attention_128": [attention(heads=2, kv_heads=1, dim=128, vdim=112, rot=48)],
    "attention_256": [attention(heads=2, kv_heads=2, dim=256, vdim=136, rot=200, window=40)],
    # layers
    "no_feed_forward": [attention(ff=0), delta(ff=0)],
    "feed_forward_sizes": [delta(ff=64), attention(ff=200), delta(ff=1)],
}
LOOPS = {
    "middle": ([delta(), attention(), delta(), attention()], (1, 3, 2)),
    "first": ([attention(), delta()], (0, 1, 3)),
    "last": ([delta(), attention()], (1, 2, 2)),
    "all": ([delta(), attention()], (0, 2, 2)),
    "once": ([delta(), attention(), delta()], (1, 2, 1)),
}


@pytest.mark.parametrize("name", list(MECHANISMS))
def test_mechanism(lm_mod, tmp_path, name):
    """One mechanism at a time: residual stream and logits of a prompt, and the same tokens in small
    portions and one by one."""
    c = Case(lm_mod, tmp_path, config(MECHANISMS[name]), seed=len(name))
    toks = tokens(c.cfg, 90, 5)
    want, taps = plain.forward(c.w, c.cfg, toks)
    for dtype in DTYPES:
        with c.open(dtype) as lm:
            s = lm.open()
            lm.tap(True)
            assert error(lm.step(s, toks, range(90)), want) < LIMIT[dtype], dtype
            got = lm.tap_read(90)
            for r in range(taps.shape[0]):
                assert np.abs(got[r] - taps[r]).max() < LIMIT[dtype] * 10 * np.abs(taps[r]).max(), (dtype, r)
            lm.tap(False)
            lm.release(s)
            for sizes in ([1], [2], [19, 2, 5, 1]):
                s = lm.open()
                assert error(feed(lm, s, toks, sizes), want) < LIMIT[dtype], (dtype, sizes)
                lm.release(s)


@pytest.mark.parametrize("name", list(LOOPS))
def test_loop(lm_mod, tmp_path, name):
    layers, loop = LOOPS[name]
    c = Case(lm_mod, tmp_path, config(layers, width=72, vocab=130, loop=loop), seed=17)
    toks = tokens(c.cfg, 70, 6)
    want, taps = plain.forward(c.w, c.cfg, toks)
    for dtype in DTYPES:
        with c.open(dtype) as lm:
            assert lm.info.runs == taps.shape[0]
            s = lm.open()
            lm.tap(True)
            assert error(lm.step(s, toks, range(70)), want) < LIMIT[dtype]
            got = lm.tap_read(70)
            for r in range(taps.shape[0]):
                assert np.abs(got[r] - taps[r]).max() < LIMIT[dtype] * 10 * np.abs(taps[r]).max(), (dtype, r)
            lm.tap(False)
            lm.release(s)
            s = lm.open()
            assert error(feed(lm, s, toks, [7, 1, 2]), want) < LIMIT[dtype]


@pytest.fixture(scope="module")
def mixed(lm_mod, tmp_path_factory):
    """Both mixers, a loop, no size a multiple of another."""
    cfg = config([delta(heads=4, kv_heads=2, dim=40, vdim=56, conv=4), attention(heads=6, kv_heads=2, dim=48, vdim=40, rot=24, window=29, keep=4),
                  delta(heads=3, kv_heads=3, dim=32, vdim=24, conv=2, ff=0)], width=168, vocab=307, loop=(1, 3, 2))
    c = Case(lm_mod, tmp_path_factory.mktemp("mixed"), cfg, seed=3)
    c.toks = tokens(cfg, 420, 8)
    c.want = plain.forward(c.w, cfg, c.toks)[0]
    return c


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[420], [2], [3, 64, 2, 31], [65, 100], [257, 1, 1, 80], [16, 17]])
def test_portions(mixed, dtype, sizes):
    with mixed.open(dtype) as lm:
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, sizes), mixed.want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("block", [1, 5, 24, 70, 130])
def test_blocks_and_ring_wraps(mixed, dtype, block):
    """A long portion runs in blocks; the ring of a windowed layer is window + block rows long and wraps
    many times."""
    with mixed.open(dtype, block_rows=block) as lm:
        assert lm.info.block_rows == block
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, [len(mixed.toks)]), mixed.want) < LIMIT[dtype]
        lm.release(s)
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, [33, 1, 8]), mixed.want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(mixed, dtype):
    """Hundreds of tokens one by one: the window passes over decoded tokens, slots of every ring are
    rewritten, the captured step is replayed."""
    with mixed.open(dtype, block_rows=16) as lm:
        s = lm.open()
        head = lm.step(s, mixed.toks[:40], range(40))
        rest = [lm.step(s, [t], [0]) for t in mixed.toks[40:]]
        assert error(np.concatenate([head] + rest), mixed.want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_wanted_places_do_not_matter(mixed, dtype):
    want = [0, 3, 64, 65, 200, 399]
    with mixed.open(dtype) as lm:
        s = lm.open()
        assert lm.step(s, mixed.toks[:10]).shape == (0, 307)
        for t in mixed.toks[10:15]:
            lm.step(s, [t])                       # nothing wanted
        got = lm.step(s, mixed.toks[15:], want)
        assert error(got, mixed.want[[w + 15 for w in want]]) < LIMIT[dtype]
        assert lm.length(s) == len(mixed.toks)


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_used_again(mixed, dtype):
    """Sequences alive side by side, given back and opened again, see nothing of one another."""
    a, b = mixed.toks[:150], mixed.toks[::-1][:90]
    want_b = plain.forward(mixed.w, mixed.cfg, b)[0]
    with mixed.open(dtype, max_seqs=2, block_rows=48) as lm:
        for _ in range(2):
            sa, sb = lm.open(), lm.open()
            with pytest.raises(RuntimeError):
                lm.open()
            got_a, got_b = [], []
            for i in range(0, 150, 15):
                got_a.append(feed(lm, sa, a[i:i + 15], [9, 1]))
                got_b.append(feed(lm, sb, b[i * 9 // 15:(i + 15) * 9 // 15], [1, 2]))
            assert error(np.concatenate(got_a), mixed.want[:150]) < LIMIT[dtype]
            assert error(np.concatenate(got_b), want_b) < LIMIT[dtype]
            lm.release(sa)
            sc = lm.open()
            assert sc == sa and lm.length(sc) == 0
            assert error(lm.step(sc, b, range(90)), want_b) < LIMIT[dtype]
            lm.release(sb)
            lm.release(sc)


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_and_kept_edges_show(lm_mod, tmp_path, dtype):
    """The edges of the window and of the kept tokens, in a prompt and in decoding: the library agrees with
    the statement, and disagrees with one whose window or kept stretch is off by one token."""
    cfg = config([attention(window=21, keep=5, ff=0, softcap=40.0)], width=96)
    c = Case(lm_mod, tmp_path, cfg, seed=9, qk_gain=2.2)
    toks = tokens(cfg, 110, 4)
    want = plain.forward(c.w, cfg, toks)[0]
    wrong = []
    for key, d in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1)):
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mixer"]["mask"][key] += d
        wrong.append(plain.forward(c.w, other, toks)[0])
    with c.open(dtype, block_rows=32) as lm:
        for sizes in ([110], [1], [2, 13]):
            s = lm.open()
            got = feed(lm, s, toks, sizes)
            lm.release(s)
            assert error(got, want) < LIMIT[dtype]
            for x in wrong:
                assert error(got, x) > 0.05


def test_far_key_among_hundreds(lm_mod, tmp_path):
    """One key far back outweighs hundreds of others: keys read one half of the stream, queries the other,
    and the last tokens' query half is the far token's key half. In a prompt, at portion borders and in
    decoding."""
    W, far, asks = 96, 3, 7
    cfg = config([attention(window=0, rot=0, softcap=0, scale=0.5, heads=2, kv_heads=1, ff=0)], width=W)
    c = Case(lm_mod, tmp_path, cfg, seed=21)
    w = c.w
    for n in ("q", "k"):
        w[f"l0.mix.{n}.norm"][:] = 1.5
    w["l0.mix.k"][:, W // 2:] = 0.0
    w["l0.mix.q"][:] = np.concatenate([w["l0.mix.k"][:, W // 2:], w["l0.mix.k"][:, :W // 2]], axis=1).tolist() * 2
    w["embed"][asks, W // 2:] = w["embed"][far, :W // 2]
    c.rewrite()
    w = c.w
    filler = [t for t in tokens(cfg, 700, 2) if t not in (far, asks)]
    toks = filler[:30] + [far] + filler[30:620] + [asks, asks]
    want = plain.forward(w, cfg, toks)[0]
    gone = plain.forward(w, cfg, toks[:30] + filler[:1] + toks[31:])[0]
    for dtype in DTYPES:
        with c.open(dtype, block_rows=256) as lm:
            for sizes in ([len(toks)], [31, 64, 2, 200], [600] + [1] * 30):
                s = lm.open()
                got = feed(lm, s, toks, sizes)
                lm.release(s)
                assert error(got, want) < LIMIT[dtype]
                assert error(got[-2:], gone[-2:]) > 0.05


def test_positions_keep_their_precision(lm_mod, tmp_path):
    """Rotation by large positions, kept tokens at their true distance."""
    cfg = config([attention(window=24, keep=2, base=100000.0, rot=32, ff=0)], width=64)
    c = Case(lm_mod, tmp_path, cfg, seed=2)
    toks = tokens(cfg, 1500, 3)
    want = plain.forward(c.w, cfg, toks)[0]
    for dtype in DTYPES:
        with c.open(dtype, block_rows=512) as lm:
            s = lm.open()
            assert error(feed(lm, s, toks, [1400, 1, 1, 98]), want) < LIMIT[dtype]


def test_long_memory_of_the_state(lm_mod, tmp_path):
    """Heads that hardly forget, over many chunks of a prompt and through decoding."""
    cfg = config([delta(heads=2, kv_heads=1, dim=64, vdim=64, conv=4, ff=0)], width=64)
    c = Case(lm_mod, tmp_path, cfg, seed=12)
    c.w["l0.mix.A_log"][:] = (-7.0, -4.0)
    c.rewrite()
    toks = tokens(cfg, 700, 3)
    want = plain.forward(c.w, cfg, toks)[0]
    for dtype in DTYPES:
        with c.open(dtype) as lm:
            for sizes in ([700], [64, 63, 65, 2], [630] + [1] * 70):
                s = lm.open()
                assert error(feed(lm, s, toks, sizes), want) < LIMIT[dtype]
                lm.release(s)


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(mixed, dtype):
    """The device-resident loop picks what the statement picks (where its choice is not a near tie), and
    what stepping token by token picks."""
    prompt, n = mixed.toks[:37], 24
    with mixed.open(dtype) as lm:
        s = lm.open()
        got = lm.generate(s, prompt, n)
        assert lm.length(s) == len(prompt) + n - 1
        # a second stretch continues the same sequence
        more = lm.generate(s, got[-1:], 10)
        lm.release(s)
        s = lm.open()
        nxt, stepped = lm.step(s, prompt, [-1])[0], []
        for _ in range(n + 10):
            stepped.append(int(np.argmax(nxt)))
            nxt = lm.step(s, [stepped[-1]], [0])[0]
        lm.release(s)
        assert got + more == stepped
        # one token at a time from the very first
        s = lm.open()
        assert lm.generate(s, prompt[:1], 1) == [int(np.argmax(mixed.want[0]))]
    logits = plain.forward(mixed.w, mixed.cfg, prompt + got + more)[0][len(prompt) - 1:-1]
    for row, t in zip(logits, got + more):
        assert row[t] > row.max() - 1e-2 * np.std(row)


def test_refusals(mixed, lm_mod, tmp_path):
    with mixed.open("bfloat16", max_tokens=64) as lm:
        s = lm.open()
        for bad in ([307], [-1], []):
            with pytest.raises(RuntimeError):
                lm.step(s, bad, [])
        with pytest.raises(RuntimeError):
            lm.step(s, mixed.toks[:65], [])
        with pytest.raises(RuntimeError):
            lm.step(s + 1, [1], [])
        with pytest.raises(RuntimeError):
            lm.step(s, [1, 2], [1, 0])
        assert lm.length(s) == 0
        assert error(lm.step(s, mixed.toks[:64], range(64)), mixed.want[:64]) < LIMIT["bfloat16"]
    w = weights(mixed.cfg, 3)
    del w["l1.mix.k.norm"]
    with pytest.raises(RuntimeError, match="l1.mix.k.norm"):
        lm_mod.LanguageModel(write_folder(tmp_path / "a", mixed.cfg, w))
    w = weights(mixed.cfg, 3)
    w["l0.mlp.up"] = w["l0.mlp.up"][:-1]
    with pytest.raises(RuntimeError, match="l0.mlp.up"):
        lm_mod.LanguageModel(write_folder(tmp_path / "b", mixed.cfg, w))


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(mixed, dtype, tmp_path):
    """bin/trace_run: steps on standard input, logits in files, one answer per step."""
    t = mixed.toks
    steps = [[{"id": "a", "tokens": t[:50], "want": [49, 0]}], [{"id": "a", "tokens": t[50:51], "want": [0]}],
             [{"id": "a", "tokens": t[51:60], "want": []}], [{"id": "b", "tokens": t[:3], "want": [2]}]]
    lines = [json.dumps({"step": i, "entries": e, "end": ["a"] if i == 2 else []}) for i, e in enumerate(steps)]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", mixed.folder, "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "100"], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    for i, rows in ((0, [49, 0]), (1, [50]), (3, [2])):
        got = np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(len(rows), -1)
        assert error(got, mixed.want[rows]) < LIMIT[dtype]
    assert not (tmp_path / "2.f32").exists()
