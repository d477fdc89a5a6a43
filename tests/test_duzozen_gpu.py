"""GPU tests of the Duzozen model: every mechanism alone and the whole model against the plain implementation of
plain_lm.py. fp32: 3e-5 normwise on logits (fp32 sums against float64). bf16: 4 % of the logits' own rms at nine
positions in ten: random routers make close calls, and where bf16 rounding turns one the logits differ visibly. Whatever
depends on a place (windows, rings, portions) is held to the sharp bound in fp32, and in bf16 by tests without a router."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import _duzozen as Z
import plain_lm as P
from _util import normwise

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
TOL = {"float32": 3e-5, "bfloat16": 4e-2}


@pytest.fixture(scope="module")
def D():
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    from ytensor_b200 import duzozen
    return duzozen


def dev(a, dtype=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).cuda()
    return t if dtype is None else t.to(dtype)


def ids(a):
    return dev(np.asarray(a, np.int32).reshape(1, -1))


def rms_error(got, want, quantile=1.0):
    """Over the positions' rms errors, relative to the rms of all logits."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    e = np.sqrt(((got - want) ** 2).mean(-1)).reshape(-1)
    return float(np.quantile(e, quantile) / np.sqrt((want ** 2).mean()))


def close(got, want, dtype):
    if dtype == "float32":
        assert normwise(got, want) < TOL[dtype]
    else:
        assert rms_error(got, want, 0.9) < TOL[dtype]


def same(a, b, dtype):
    """Two ways of computing the same logits on the device."""
    assert rms_error(a, b) < 2e-5 if dtype == "float32" else rms_error(a, b, 0.9) < TOL[dtype]


def model(D, cfg, w, dtype="float32", **kw):
    m = D.DuzozenForCausalLM(cfg, dtype=dtype, **kw)
    m.load_weights(w)
    return m


def run(m, toks, cuts):
    """Logits of every position, the tokens cut into portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(m.forward_at(ids(toks[at:at + n]), range(n)).cpu().numpy())
        at, i = at + n, i + 1
    return np.concatenate(out)


# ---------------------------------------------------------------- mechanisms
def attention_case(D, dtype, T, pos0, H, G, d, dv, window, cap, ring, spike=True, seed=0):
    """Queries at pos0 .. pos0 + T - 1 over a ring; single keys at and around the window's edge get a large score."""
    from ytensor_b200 import _lib
    rng = np.random.default_rng(seed)
    S = pos0 + T
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((S, G, d)) * 0.3, rng.standard_normal((S, G, dv))
    if spike:  # every 7th query points at the last key inside its window, the next one at the first outside
        for t in range(0, T, 7):
            for u, off in ((t, window - 1), (t + 1, window)):
                j = pos0 + u - off
                if window and u < T and j >= 0:
                    q[u, :, :] *= 0.2
                    for h in range(H):
                        q[u, h] += k[j, h // (H // G)] * 6
    tt = torch.float32 if dtype == "float32" else torch.bfloat16
    qd, kd, vd = dev(q, tt), dev(k, tt), dev(v, tt)
    kr = torch.zeros(G, ring, d, dtype=tt, device="cuda")
    vr = torch.zeros(G, ring, dv, dtype=tt, device="cuda")
    for p in range(max(0, S - ring), S):
        kr[:, p % ring], vr[:, p % ring] = kd[p], vd[p]
    o = torch.empty(T, H, dv, dtype=tt, device="cuda")
    import ctypes as C
    st = lambda *x: C.cast((C.c_int64 * 3)(*x), C.c_void_p)  # noqa: E731
    scale = 0.7 * d ** -0.5
    _lib.check(_lib.lib().ytcuda_window_attn_fwd(
        _lib.F32 if dtype == "float32" else _lib.BF16, qd.data_ptr(), kr.data_ptr(), vr.data_ptr(), o.data_ptr(), 1, G,
        H // G, T, d, dv, st(T * H * d, d, H * d), st(G * ring * d, ring * d, d), st(G * ring * dv, ring * dv, dv),
        st(T * H * dv, dv, H * dv), pos0, window, ring, scale, cap, torch.cuda.current_stream().cuda_stream))
    want = P.attention(qd.double().cpu().numpy(), kd.double().cpu().numpy(), vd.double().cpu().numpy(), scale,
                       cap or None, window or None)
    err = normwise(o.float().cpu().numpy(), want)
    assert err < (1e-5 if dtype == "float32" else 1.5e-2), (err, T, pos0, window, cap)


@pytest.mark.parametrize("dtype,d,dv", [("float32", 20, 36), ("float32", 64, 64), ("bfloat16", 24, 40),
                                        ("bfloat16", 64, 64), ("bfloat16", 128, 128)])
def test_window_attention(D, dtype, d, dv):
    for T, pos0, H, G, window, cap, ring in [
            (40, 0, 2, 2, 9, 15.0, 128), (2, 200, 3, 1, 72, 15.0, 384), (130, 127, 4, 2, 128, 0.0, 384),
            (150, 300, 2, 1, 1, 25.0, 256), (140, 250, 6, 2, 129, 60.0, 512), (33, 1000, 2, 2, 200, 40.0, 384),
            (257, 0, 1, 1, 64, 5.0, 384), (20, 100, 2, 2, 0, 0.0, 128), (131, 60, 2, 1, 0, 20.0, 256),
            (64, 64, 2, 2, 127, 15.0, 256), (3, 126, 2, 2, 3, 15.0, 256)]:
        attention_case(D, dtype, T, pos0, H, G, d, dv, window, cap, ring)


def test_window_attention_refuses_a_ring_that_is_too_short(D):
    with pytest.raises(ValueError):
        attention_case(D, "float32", 100, 0, 1, 1, 16, 16, 0, 0.0, 64, spike=False)


@pytest.mark.parametrize("experts,identity,top,count,keep", [(8, 4, 4, 3, 2), (7, 2, 3, 1, 1), (60, 4, 8, 8, 3), (5, 0, 5, 1, 1),
                                                             (40, 40, 6, 40, 7), (3, 9, 2, 4, 1), (1, 0, 1, 1, 1)])
def test_router(D, experts, identity, top, count, keep):
    from ytensor_b200 import _lib
    rng = np.random.default_rng(experts + top)
    n, rows = experts + identity, 53
    z = (rng.standard_normal((rows, n)) * 1.5).astype(np.float32)
    corr = (rng.standard_normal(n) * 0.3 - 0.6).astype(np.float32)  # most choice scores are negative
    ch = torch.empty(rows, top, dtype=torch.int32, device="cuda")
    rk, w = torch.empty_like(ch), torch.empty(rows, top, device="cuda")
    cnt = torch.zeros(experts, dtype=torch.int32, device="cuda")
    zd, cd = dev(z), dev(corr)
    _lib.check(_lib.lib().ytcuda_moe_route(zd.data_ptr(), n, cd.data_ptr(), rows, experts, identity, top, count, keep, 0,
                                           ch.data_ptr(), w.data_ptr(), rk.data_ptr(), cnt.data_ptr(), None))
    got, gw, grk = ch.cpu().numpy(), w.cpu().numpy(), rk.cpu().numpy()
    for t in range(rows):
        want, ww = P.route(z[t].astype(np.float64), corr.astype(np.float64), top, count, keep)
        assert got[t].tolist()[:len(want)] == want and (got[t, len(want):] == -1).all()
        assert np.abs(gw[t, :len(want)] - ww).max() < 1e-6
    for e in range(experts):  # the ranks of an expert's tokens are 0 .. count - 1
        assert sorted(grk[got == e].tolist()) == list(range(int(cnt[e])))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [44, 1024, 5000])
def test_residual_norm(D, dtype, width):
    from ytensor_b200 import _lib
    rng = np.random.default_rng(width)
    ld, rows, eps = (width + 7) // 8 * 8, 5, 1e-3

    def padded(a):
        out = np.zeros(a.shape[:-1] + (ld,), np.float32)
        out[..., :width] = a
        return out

    x, y, a, b = (padded(rng.standard_normal(s).astype(np.float32)) for s in ((rows, width), (rows, width), (width,), (width,)))
    tt = torch.float32 if dtype == "float32" else torch.bfloat16
    xd, yd, ad, bd, h = dev(x), dev(y), dev(a), dev(b), torch.empty(rows, ld, dtype=tt, device="cuda")
    code = _lib.F32 if dtype == "float32" else _lib.BF16
    _lib.check(_lib.lib().ytcuda_residual_norm(xd.data_ptr(), yd.data_ptr(), ad.data_ptr(), bd.data_ptr(), h.data_ptr(), code,
                                               rows, width, ld, eps, None))
    w64 = lambda t: t[..., :width].astype(np.float64)  # noqa: E731
    wx = w64(x) + P.rms_norm(w64(y), w64(a), eps)
    assert normwise(xd.cpu().numpy()[:, :width], wx) < 1e-6
    assert normwise(h.float().cpu().numpy()[:, :width], P.rms_norm(wx, w64(b), eps)) < (1e-6 if dtype == "float32" else 5e-3)
    assert not xd[:, width:].any() and not h[:, width:].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("m,n,k", [(3, 40, 24), (130, 300, 264), (700, 512, 1024), (300, 46, 72)])
def test_linear_with_activation(D, dtype, m, n, k):
    from ytensor_b200 import _lib
    rng = np.random.default_rng(m)
    tt = torch.float32 if dtype == "float32" else torch.bfloat16
    code = _lib.F32 if dtype == "float32" else _lib.BF16
    x, w = dev(rng.standard_normal((m, k)), tt), dev(rng.standard_normal((n, k)) / np.sqrt(k) * 1.5, torch.bfloat16)
    z = x.double().cpu().numpy() @ w.double().cpu().numpy().T
    for act, want in ((0, z), (1, P.gelu_erf(z)), (2, P.silu(z[:, ::2]) * z[:, 1::2])):
        y = torch.empty(m, want.shape[1], dtype=tt, device="cuda")
        _lib.check(_lib.lib().ytcuda_linear_act(code, act, x.data_ptr(), k, w.data_ptr(), y.data_ptr(), want.shape[1], m, n, k,
                                                0, 0.0, None, 1, torch.cuda.current_stream().cuda_stream))
        assert normwise(y.float().cpu().numpy(), want) < (2e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_grouped_linear(D, dtype):
    from ytensor_b200 import _lib
    rng = np.random.default_rng(1)
    E, n, k, blocks = 4, 88, 136, [2, 0, -1, 3, 3, 1]
    tt = torch.float32 if dtype == "float32" else torch.bfloat16
    code = _lib.F32 if dtype == "float32" else _lib.BF16
    m = 128 * len(blocks)
    x, w = dev(rng.standard_normal((m, k)), tt), dev(rng.standard_normal((E, n, k)) / np.sqrt(k), torch.bfloat16)
    bg = dev(np.asarray(blocks, np.int32))
    for act in (0, 2):
        cols = n // 2 if act == 2 else n
        y = torch.full((m, cols), 7.0, dtype=tt, device="cuda")
        _lib.check(_lib.lib().ytcuda_linear_act(code, act, x.data_ptr(), k, w.data_ptr(), y.data_ptr(), cols, m, n, k,
                                                0, 0.0, bg.data_ptr(), E, torch.cuda.current_stream().cuda_stream))
        got = y.float().cpu().numpy()
        for i, e in enumerate(blocks):
            rows = slice(128 * i, 128 * i + 128)
            if e < 0:
                assert (got[rows] == 7.0).all()  # passed over
                continue
            z = x[rows].double().cpu().numpy() @ w[e].double().cpu().numpy().T
            want = z if act == 0 else P.silu(z[:, ::2]) * z[:, 1::2]
            assert normwise(got[rows], want) < (2e-6 if dtype == "float32" else 5e-3)


# ---------------------------------------------------------------- the model
def longest(cfg):
    return max(x.window for x in cfg.layers)


@pytest.fixture(scope="module")
def cases():
    out = {}
    for name, make in Z.CONFIGS.items():
        cfg = make()
        w = Z.weights(cfg, seed=len(name))
        toks = np.random.default_rng(5).integers(0, cfg.vocab, 60 + longest(cfg)).tolist()
        out[name] = (cfg, w, toks, P.forward(cfg.to_dict(), Z.floats(w), toks))
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_prompt_portions_and_decoding(D, cases, name, dtype):
    """The whole prompt in one call, in portions down to two tokens, and token by token: the same logits everywhere, also
    in the first positions and on both sides of every window's edge; with rings that are used over and over (chunk 32)."""
    cfg, w, toks, want = cases[name]
    whole = None
    for chunk, cuts in ((4096, [len(toks)]), (32, [len(toks)]), (32, [3, 2, 7, 2, 31, 1, 2, 40]), (4096, [2]), (32, [5, 1])):
        m = model(D, cfg, w, dtype, max_tokens=len(toks), chunk=chunk)
        got = run(m, toks, cuts)
        close(got, want, dtype)
        whole = got if whole is None else whole
        same(got, whole, dtype)
        assert m.get_kv_cache_len() == len(toks)
        m.check_status()
        m.close()


@pytest.mark.parametrize("d,dv,heads,kv", [(64, 64, 4, 4), (128, 128, 4, 1), (40, 24, 6, 3), (136, 40, 2, 1)])
def test_bf16_without_a_router(D, d, dv, heads, kv):
    """Dense layers in bf16: every position, in every portion, within 4 % - tensor-core attention with both tile widths,
    padded heads, and head dims beyond the tensor-core tiles."""
    cfg = Z.config([Z.layer(heads, kv, d, dv, window=w, cap=c, ff=96) for w, c in ((50, 20.0), (129, 60.0), (0, 0.0))],
                   width=72, vocab=110)
    w = Z.weights(cfg, seed=d, qk_gain=1.5)
    toks = np.random.default_rng(6).integers(0, cfg.vocab, 300).tolist()
    want = P.forward(cfg.to_dict(), Z.floats(w), toks)
    for cuts in ([300], [130, 2, 3, 65, 1]):
        m = model(D, cfg, w, "bfloat16", max_tokens=300, chunk=64)
        got = run(m, toks, cuts)
        assert rms_error(got, want) < TOL["bfloat16"]
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_decode_kernels_match_the_operator_path(D, cases, name, dtype):
    cfg, w, toks, _ = cases[name]
    a, b = (model(D, cfg, w, dtype, max_tokens=len(toks), chunk=32) for _ in range(2))
    b.set_decode_path(1)
    from ytensor_b200 import _lib
    ga, gb = run(a, toks, [11, 1]), run(b, toks, [11, 1])
    same(ga, gb, dtype)
    n0 = _lib.lib().ytcuda_launch_count()
    a.reset_kv_cache()
    a.forward(ids(toks[:1]))
    used = _lib.lib().ytcuda_launch_count() - n0  # (one more than the step's kernels: the position word)
    assert used <= 2 + sum(3 if x.mlp == 0 else 5 if x.mlp == 1 else 6 for x in cfg.layers)
    a.close()
    b.close()


def test_long_decoding_far_past_the_ring(D):
    """Far more tokens than a ring holds, decoded one by one; the oracle sees the whole sequence."""
    cfg = Z.config([Z.layer(2, 1, 16, 24, window=33, ff=24),
                    Z.layer(2, 1, 16, 24, window=10, mlp="moe", ff=16, experts=4, identity=2, top=2, groups=3, keep=2)],
                   width=32, vocab=40)
    w = Z.weights(cfg, seed=3)
    toks = np.random.default_rng(1).integers(0, cfg.vocab, 620).tolist()
    want = P.forward(cfg.to_dict(), Z.floats(w), toks)
    m = model(D, cfg, w, "float32", max_tokens=1000, chunk=16)  # rings of 256 positions
    got = run(m, toks, [50, 1])
    close(got, want, "float32")
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_key_that_stands_out_is_seen_up_to_the_edge_and_not_beyond(D, dtype):
    """One layer with one-hot tokens: token 1's key answers token 2's query alone, so token 2's logits tell whether a
    token 1 that lies `gap` positions back is seen. Prompt and decoding, gaps just inside and just outside the window, at
    tile borders of the ring."""
    width, vocab = 16, 8
    for window in (4, 100, 128, 129):
        cfg = Z.config([Z.layer(1, 1, 8, 8, window=window, cap=20.0, scale=1.0, v_mix=False, mlp=None)], width=width, vocab=vocab)
        f = {n: np.zeros(s, np.float32) for n, s in cfg.tensor_shapes().items()}
        for n in ("l0.norm1", "l0.norm1b", "final.norm"):
            f[n][:] = 1
        f["embed"][np.arange(vocab), np.arange(vocab)] = 1
        f["l0.mix.q"][0, 2] = 5          # token 2 asks along channel 0 ...
        f["l0.mix.k"][0, 1] = 1          # ... token 1 answers
        f["l0.mix.v"][1, 1] = f["l0.mix.v"][2, 3] = 1
        f["l0.mix.o"][9, 1] = f["l0.mix.o"][10, 2] = 1
        f["head"][1, 9] = f["head"][3, 10] = 3
        w = {n: (Z.f32_to_bf16_bits(a)) for n, a in f.items()}
        m = model(D, cfg, w, dtype, max_tokens=700, chunk=64)
        for at in (0, 126, 127, 128, 255):
            for gap in (window - 1, window):
                toks = [3] * at + [1] + [3] * (gap - 1) + [2]
                plain = P.forward(cfg.to_dict(), Z.floats(w), toks)[-1]
                seen = plain[1] > plain[3]
                assert seen == (gap == window - 1)
                for cuts in ([len(toks)], [len(toks) - 1, 1], [max(1, len(toks) - 2), 2]):
                    m.reset_kv_cache()
                    got = run(m, toks, cuts)[-1]
                    assert rms_error(got[None], plain[None]) < (1e-4 if dtype == "float32" else 2e-2)
        m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_cache_that_is_used_again_leaves_no_trace(D, cases, dtype):
    cfg, w, toks, want = cases["mixed"]
    other = np.random.default_rng(9).integers(0, cfg.vocab, 75).tolist()
    m = model(D, cfg, w, dtype, max_tokens=len(toks), chunk=32)
    first = run(m, toks, [9, 1, 13])
    m.reset_kv_cache()
    assert m.get_kv_cache_len() == 0
    run(m, other, [75])
    m.reset_kv_cache()
    again = run(m, toks, [9, 1, 13])
    assert np.array_equal(first, again)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_batch_equals_each_sequence_alone(D, cases, dtype):
    cfg, w, _, _ = cases["mixed"]
    rng = np.random.default_rng(2)
    toks = rng.integers(0, cfg.vocab, (3, 70)).astype(np.int32)
    b = model(D, cfg, w, dtype, batch=3, max_tokens=70, chunk=32)
    got = [b.forward(dev(toks[:, :50])).cpu().numpy()] + [b.forward(dev(toks[:, t:t + 1])).cpu().numpy() for t in range(50, 70)]
    b.close()
    m = model(D, cfg, w, dtype, max_tokens=70)
    for s in range(3):
        m.reset_kv_cache()
        alone = run(m, toks[s].tolist(), [50, 1])[49:]
        same(np.stack([g[s] for g in got]), alone, dtype)
    m.close()


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_greedy_generation(D, cases, name):
    cfg, w, toks, _ = cases[name]
    prompt = toks[:13]
    want = P.greedy(cfg.to_dict(), Z.floats(w), prompt, 24)
    m = model(D, cfg, w, "float32", max_tokens=64)
    got = m.generate_greedy(ids(prompt), 24).cpu().numpy()[0].tolist()
    assert got == want
    m.reset_kv_cache()
    assert m.generate_topk(ids(prompt), 24, k=1).cpu().numpy()[0].tolist() == want  # k = 1 is greedy decoding
    m.reset_kv_cache()
    a = m.generate_topk(ids(prompt), 12, k=5, seed=3).cpu().numpy()
    m.reset_kv_cache()
    assert np.array_equal(a, m.generate_topk(ids(prompt), 12, k=5, seed=3).cpu().numpy())
    m.close()


def save(folder, cfg, w):
    from ytensor_b200.safetensors import write_safetensors
    folder.mkdir(exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg.to_dict()))
    write_safetensors(folder / "model.safetensors", w)


def test_registry_command_line_and_trace(D, cases, tmp_path):
    from ytensor_b200.registry import load_model
    cfg, w, toks, want = cases["odd"]
    save(tmp_path / "m", cfg, w)
    m = load_model(tmp_path / "m", dtype="float32", max_tokens=64)
    assert isinstance(m, D.DuzozenForCausalLM)
    greedy = m.generate_greedy(ids(toks[:9]), 8).cpu().numpy()[0].tolist()
    m.close()
    env = dict(os.environ, PYTHONPATH=str(ROOT))
    r = subprocess.run([sys.executable, "-m", "ytensor_b200", "generate", "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--tokens", ",".join(map(str, toks[:9])), "--steps", "8"], capture_output=True, text=True, env=env,
                       timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()[-1].split(",")] == greedy
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:20], "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[20:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[21:23], "want": [1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}], "end": []}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    for step, places in ((0, [19, 3]), (2, [22]), (3, [0])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, cfg.vocab)
        close(got, want[places], "float32")
    assert not (tmp_path / "1.f32").exists()


def test_bad_calls_are_refused(D, cases):
    cfg, w, toks, _ = cases["odd"]
    m = model(D, cfg, w, max_tokens=20)
    with pytest.raises(ValueError):
        m.forward(ids(toks[:21]))        # longer than the sequence may be
    with pytest.raises(ValueError):
        m.forward_at(ids(toks[:5]), [5])
    m.close()
    with pytest.raises(ValueError):
        D.DuzozenForCausalLM(Z.config([Z.layer(5, 2)]))
    with pytest.raises(ValueError):
        D.DuzozenForCausalLM(cfg, dtype="float16")
    with pytest.raises(ValueError):
        model(D, cfg, dict(w, head=w["head"][:-1]))
