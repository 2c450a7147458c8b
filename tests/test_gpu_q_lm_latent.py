"""Latent attention, shared latents, parallel layers and mixtures of experts (the Bupozen design) on the GPU
against the plain statement (lm_plain.py), through the library's own step function, slots and
generation loop."""
import json
import os
import subprocess

import numpy as np
import pytest

import lm_plain as plain
from lm_models import DTYPES, LIMIT, Case, config, error, feed, latent, tokens, weights, write_folder

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def lm_mod(pkg):
    return pkg


MECHANISMS = {
    # attention alone
    "latent": [latent(ff=0)],
    "every_key": [latent(window=0, ff=0)],
    "window_one": [latent(window=1, ff=0)],
    "window_two": [latent(window=2, ff=0)],
    "window_past_the_prompt": [latent(window=500, ff=0)],
    "no_rotated_part": [latent(rot_dim=0, ff=0)],
    "rotation_of_a_part": [latent(rot_dim=16, rot=6, ff=0)],
    "rotation_base": [latent(rot_dim=24, base=40.0, scale=0.5, ff=0)],
    "one_head": [latent(heads=1, ff=0)],
    "many_heads": [latent(heads=21, dim=8, vdim=8, ff=0)],
    "odd_sizes": [latent(heads=3, dim=13, rot_dim=6, vdim=11, kv_rank=37, q_rank=29, ff=0)],
    "tiny_latents": [latent(heads=2, kv_rank=8, q_rank=1, dim=8, vdim=8, ff=0)],
    "rank_not_in_eights": [latent(kv_rank=44, rot_dim=4, ff=0)],
    "heads_of_192": [latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=264, q_rank=160, scale=0.09, ff=0)],
    "heads_of_96": [latent(heads=3, dim=80, rot_dim=16, vdim=72, kv_rank=136, q_rank=100, ff=0)],
    "heads_too_large_to_write_out": [latent(heads=2, dim=200, rot_dim=16, vdim=136, kv_rank=96, scale=0.08, ff=0)],
    "rank_of_512": [latent(heads=2, dim=32, rot_dim=64, vdim=32, kv_rank=512, ff=0)],
    "rank_of_1032": [latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=1032, ff=0)],
    # feed-forward beside it
    "dense": [latent()],
    "dense_sizes": [latent(ff=1), latent(ff=200), latent(ff=67)],
    "experts": [latent(ff=40, experts=6, top=2)],
    "experts_one_chosen": [latent(ff=33, experts=5, top=1)],
    "experts_all_chosen": [latent(ff=24, experts=3, top=3)],
    "experts_one": [latent(ff=72, experts=1, top=1)],
    "experts_many": [latent(ff=16, experts=45, top=7)],
    "experts_large": [latent(ff=260, experts=4, top=2)],
    # another layer's latents
    "shared": [latent(), latent(kv_from=0)],
    "shared_far_back": [latent(), latent(kv_rank=32), latent(kv_from=0, ff=0), latent(kv_from=1, kv_rank=32), latent(kv_from=0)],
    "shared_longer_window": [latent(window=5), latent(kv_from=0, window=33), latent(kv_from=0, window=1)],
    "shared_every_key": [latent(window=7), latent(kv_from=0, window=0)],
    "shared_other_heads": [latent(heads=2, dim=32, vdim=24), latent(kv_from=0, heads=5, dim=16, vdim=48, q_rank=30, scale=0.4)],
    "shared_by_experts": [latent(ff=30, experts=4), latent(kv_from=0, ff=50, experts=7, top=3)],
}


@pytest.mark.parametrize("name", list(MECHANISMS))
def test_mechanism(lm_mod, tmp_path, name):
    """One mechanism at a time: residual stream and logits of a prompt, and the same tokens in small
    portions and one by one."""
    c = Case(lm_mod, tmp_path, config(MECHANISMS[name]), seed=len(name))
    toks = tokens(c.cfg, 90, 5)
    want, taps = plain.forward(c.w, c.cfg, toks)
    for dtype in DTYPES:
        with c.open(dtype, block_rows=96) as lm:
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


@pytest.mark.parametrize("width,vocab,eps,n", [(64, 50, 1e-3, 70), (130, 333, 1e-6, 70), (77, 31, 1e-5, 70), (400, 90, 1e-5, 300), (633, 70, 1e-4, 270)])
def test_stream_sizes(lm_mod, tmp_path, width, vocab, eps, n):
    c = Case(lm_mod, tmp_path, config([latent(ff=0, window=9), latent(ff=350), latent(ff=170, experts=5)], width=width, vocab=vocab, eps=eps), seed=2)
    toks = tokens(c.cfg, n, 5)
    want = plain.forward(c.w, c.cfg, toks)[0]
    for dtype in DTYPES:
        with c.open(dtype) as lm:
            for sizes in ([n], [30, 1, 3]):
                s = lm.open()
                assert error(feed(lm, s, toks, sizes), want) < LIMIT[dtype], (dtype, sizes)
                lm.release(s)


@pytest.fixture(scope="module")
def mixed(lm_mod, tmp_path_factory):
    """Dense, mixed and absent feed-forwards, own and shared latents, three windows."""
    cfg = config([latent(window=31, ff=88), latent(window=47, kv_from=0, ff=40, experts=7, top=3), latent(heads=6, kv_rank=72, window=0, ff=0),
                  latent(heads=2, kv_rank=72, kv_from=2, window=12, ff=150)], width=168, vocab=307)
    c = Case(lm_mod, tmp_path_factory.mktemp("latent"), cfg, seed=3)
    c.toks = tokens(cfg, 420, 8)
    c.want = plain.forward(c.w, cfg, c.toks)[0]
    return c


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [[420], [2], [3, 64, 2, 31], [65, 100], [257, 1, 1, 80], [16, 17, 4, 5], [256, 128, 36]])
def test_portions(mixed, dtype, sizes):
    with mixed.open(dtype) as lm:
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, sizes), mixed.want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("block", [1, 5, 24, 70, 130])
def test_blocks_and_ring_wraps(mixed, dtype, block):
    """A long portion runs in blocks; a windowed layer's ring is as long as the longest window that reads it
    plus a block, and wraps many times."""
    with mixed.open(dtype, block_rows=block, max_tokens=430) as lm:
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, [len(mixed.toks)]), mixed.want) < LIMIT[dtype]
        lm.release(s)
        s = lm.open()
        assert error(feed(lm, s, mixed.toks, [33, 1, 8]), mixed.want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(mixed, dtype):
    """Hundreds of tokens one by one: windows pass over decoded tokens, the captured step is replayed."""
    with mixed.open(dtype, block_rows=40) as lm:
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
            lm.step(s, [t])
        got = lm.step(s, mixed.toks[15:], want)
        assert error(got, mixed.want[[w + 15 for w in want]]) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_used_again(mixed, dtype):
    """Sequences of unequal length alive side by side, given back and opened again, see nothing of one another."""
    a, b = mixed.toks[:150], mixed.toks[::-1][:90]
    want_b = plain.forward(mixed.w, mixed.cfg, b)[0]
    with mixed.open(dtype, max_seqs=2, block_rows=48) as lm:
        for _ in range(2):
            sa, sb = lm.open(), lm.open()
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
def test_planted_mistakes_show(lm_mod, tmp_path, dtype):
    """The library agrees with the statement, in a prompt and in decoding, and disagrees with one whose window is
    off by one token, whose shared latents come from another layer, whose rotation, scale, routing or eps
    differs."""
    cfg = config([latent(window=21, scale=0.7, ff=50), latent(window=21, kv_from=0, scale=0.7, ff=40, experts=6, top=3),
                  latent(window=21, scale=0.7, ff=0), latent(window=30, kv_from=2, scale=0.7, ff=0)], width=96, eps=0.05)
    c = Case(lm_mod, tmp_path, cfg, seed=9, qk_gain=2.2)
    toks = tokens(cfg, 110, 4)
    want = plain.forward(c.w, cfg, toks)[0]
    wrong = []

    def plant(change):
        other = json.loads(json.dumps(cfg))
        change(other)
        wrong.append(plain.forward(c.w, other, toks)[0])

    for d in (1, -1):
        plant(lambda o: o["layers"][0]["mixer"]["mask"].update(size=21 + d))
        plant(lambda o: o["layers"][3]["mixer"]["mask"].update(size=30 + d))
    plant(lambda o: o["layers"][3]["mixer"].update(kv_from=0))
    plant(lambda o: o["layers"][1]["mlp"]["router"].update(top=2))
    plant(lambda o: o["layers"][0]["mixer"]["rot"].update(base=2000.0))
    plant(lambda o: o["layers"][2]["mixer"].update(scale=0.6))
    plant(lambda o: o["norm"].update(eps=0.1))
    # the last window's worth of positions is compared: earlier ones see no edge
    with c.open(dtype, block_rows=32) as lm:
        for sizes in ([110], [1], [2, 13]):
            s = lm.open()
            got = feed(lm, s, toks, sizes)
            lm.release(s)
            assert error(got, want) < LIMIT[dtype]
            for i, x in enumerate(wrong):
                assert error(got[40:], x[40:]) > 0.02, (sizes, i)


@pytest.mark.parametrize("shared", [False, True])
def test_far_key_among_hundreds(lm_mod, tmp_path, shared):
    """One key far back outweighs hundreds of others: latents read one half of the stream, queries the other, and the
    last tokens' query half is the far token's key half. In a prompt, at portion borders and in decoding;
    also where the attention reads another layer's latents."""
    W, far, asks = 96, 3, 7
    layers = [latent(window=0, heads=2, dim=32, kv_rank=40, q_rank=40, scale=0.6, ff=0)]
    if shared:
        layers = [latent(window=4, heads=1, kv_rank=40, ff=0)] + layers
        layers[1]["mixer"]["kv_from"] = 0
    cfg = config(layers, width=W)
    c = Case(lm_mod, tmp_path, cfg, seed=21)
    w, p = c.w, f"l{len(layers) - 1}.mix"
    w["l0.mix.dkv.norm"][:] = w[p + ".dq.norm"][:] = 1.25
    w["l0.mix.dkv"][:, W // 2:] = 0.0
    w[p + ".dq"][:] = np.concatenate([w["l0.mix.dkv"][:40, W // 2:], w["l0.mix.dkv"][:40, :W // 2]], axis=1)
    uq = w[p + ".uq"].reshape(2, 40, 40)                    # 32 plain and 8 rotated rows per head
    uq[:, :32] = w[p + ".uk"].reshape(2, 32, 40)
    uq[:, 32:] = 0.0
    w["embed"][asks, W // 2:] = w["embed"][far, :W // 2]
    if shared:
        w["l0.mix.o"][:] = 0.0
    c.rewrite()
    filler = [t for t in tokens(cfg, 700, 2) if t not in (far, asks)]
    toks = filler[:30] + [far] + filler[30:620] + [asks, asks]
    want = plain.forward(c.w, cfg, toks)[0]
    gone = plain.forward(c.w, cfg, toks[:30] + filler[:1] + toks[31:])[0]
    for dtype in DTYPES:
        with c.open(dtype, block_rows=256) as lm:
            for sizes in ([len(toks)], [31, 64, 2, 200], [600] + [1] * 30):
                s = lm.open()
                got = feed(lm, s, toks, sizes)
                lm.release(s)
                assert error(got, want) < LIMIT[dtype]
                assert error(got[-2:], gone[-2:]) > 0.05


def test_positions_keep_their_precision(lm_mod, tmp_path):
    """Rotation by large positions."""
    cfg = config([latent(window=24, base=100000.0, rot_dim=32, scale=0.6, ff=0)], width=64)
    c = Case(lm_mod, tmp_path, cfg, seed=2)
    toks = tokens(cfg, 1500, 3)
    want = plain.forward(c.w, cfg, toks)[0]
    for dtype in DTYPES:
        with c.open(dtype, block_rows=512) as lm:
            s = lm.open()
            assert error(feed(lm, s, toks, [1400, 1, 1, 98]), want) < LIMIT[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_experts_that_get_nothing_or_everything(lm_mod, tmp_path, dtype):
    """A router that sends every token to the same experts (more rows than a block of 128 holds), and one that sends
    tokens apart by a single stream dimension."""
    cfg = config([latent(ff=48, experts=9, top=2), latent(ff=48, experts=9, top=1)], width=72, vocab=90)
    c = Case(lm_mod, tmp_path, cfg, seed=5)
    c.w["l0.mlp.router"][:] *= 1e-3
    c.w["l0.mlp.router"][[4, 7]] = 0.0
    c.w["l0.norm1"][0] = c.w["l1.norm1"][0] = 1.0
    c.w["embed"][:, 0] = 2.0 + np.arange(90) % 2
    c.w["l0.mlp.router"][4, 0], c.w["l0.mlp.router"][7, 0] = 4.0, 3.5
    c.w["l1.mlp.router"][:, 0] = 0.0
    c.rewrite()
    toks = tokens(cfg, 300, 6)
    want = plain.forward(c.w, cfg, toks)[0]
    with c.open(dtype) as lm:
        for sizes in ([300], [140, 3, 1, 60]):
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
        more = lm.generate(s, got[-1:], 10)
        lm.release(s)
        s = lm.open()
        nxt, stepped = lm.step(s, prompt, [-1])[0], []
        for _ in range(n + 10):
            stepped.append(int(np.argmax(nxt)))
            nxt = lm.step(s, [stepped[-1]], [0])[0]
        lm.release(s)
        assert got + more == stepped
    logits = plain.forward(mixed.w, mixed.cfg, prompt + got + more)[0][len(prompt) - 1:-1]
    for row, t in zip(logits, got + more):
        assert row[t] > row.max() - 1e-2 * np.std(row)


def test_refusals(mixed, lm_mod, tmp_path):
    for i, (name, match) in enumerate((("l0.mix.dkv.norm", None), ("l1.mlp.e5.down", None), ("l1.mlp.router", None), ("l3.mix.g", None))):
        w = weights(mixed.cfg, 3)
        del w[name]
        with pytest.raises(RuntimeError, match=name):
            lm_mod.LanguageModel(write_folder(tmp_path / str(i), mixed.cfg, w))
    w = weights(mixed.cfg, 3)
    w["l2.mix.uk"] = w["l2.mix.uk"][:, :-1].copy()
    with pytest.raises(RuntimeError, match="l2.mix.uk"):
        lm_mod.LanguageModel(write_folder(tmp_path / "x", mixed.cfg, w))


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
