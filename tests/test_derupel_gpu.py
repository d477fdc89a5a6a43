"""GPU tests of the Derupel model: every mechanism alone and the whole model against the plain implementation of
plain_derupel.py. fp32: 3e-5 normwise on logits (fp32 sums against float64). bf16: 4 % of the logits' own rms at three
positions in four: random routers make close calls, and where bf16 rounding turns one the logits differ visibly, also at the
positions that remember it. Whatever
depends on a place (tiles, chunks, portions) is held to the sharp bound in fp32, and in bf16 by tests without a router."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import _derupel as Z
import plain_derupel as P
from _util import normwise
from plain_lm import rms_norm, silu

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
TOL = {"float32": 3e-5, "bfloat16": 4e-2}
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def D():
    if not torch.cuda.is_available():
        pytest.skip("no CUDA device")
    from ytensor_b200 import derupel
    return derupel


@pytest.fixture(scope="module")
def L(D):
    from ytensor_b200 import _lib
    return _lib.lib()


def dev(a, dtype=None):
    t = torch.from_numpy(np.ascontiguousarray(a)).cuda()
    return t if dtype is None else t.to(dtype)


def f64(t):
    return t.double().cpu().numpy()


def kind(dtype):
    from ytensor_b200 import _lib
    return (torch.float32, _lib.F32) if dtype == "float32" else (torch.bfloat16, _lib.BF16)


def check(status):
    from ytensor_b200 import _lib
    _lib.check(status)


def stream():
    return torch.cuda.current_stream().cuda_stream


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
        assert rms_error(got, want, 0.75) < TOL[dtype]


def same(a, b, dtype):
    """Two ways of computing the same logits on the device."""
    assert rms_error(a, b) < 2e-5 if dtype == "float32" else rms_error(a, b, 0.75) < TOL[dtype]


def model(D, cfg, w, dtype="float32", **kw):
    m = D.DerupelForCausalLM(cfg, dtype=dtype, **kw)
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


# ---------------------------------------------------------------- linear attention with a decayed state
def decayed_case(L, dtype, cuts, batch, H, d, dv, decay, path, seed=0):
    """Calls over one sequence per batch entry, cut into portions; the state is carried from call to call."""
    rng = np.random.default_rng(seed)
    tt, code = kind(dtype)
    T = sum(cuts)
    q, k, v = (dev(silu(rng.standard_normal((batch, T, H, n)) * 2), tt) for n in (d, d, dv))
    w = dev(np.asarray(decay, np.float32))
    state = torch.full((batch, H, d, dv), 1e9, device="cuda")  # what an earlier sequence left
    outs, at = [], 0
    for n in cuts:
        rows = torch.cat([t[:, at:at + n].reshape(batch, n, -1) for t in (q, k, v)], -1).contiguous()
        o = torch.empty(batch, n, H, dv, dtype=tt, device="cuda")
        e = rows.element_size()
        check(L.ytcuda_decayed_attn_fwd(code, rows.data_ptr(), rows.data_ptr() + H * d * e, rows.data_ptr() + 2 * H * d * e,
                                        rows.shape[-1], o.data_ptr(), state.data_ptr(), w.data_ptr(), batch, n, H, d, dv,
                                        int(at == 0), path, stream()))
        outs.append(f64(o))
        at += n
    got = np.concatenate(outs, 1)
    for b in range(batch):
        want, end = P.decayed_attention(f64(q[b]), f64(k[b]), f64(v[b]), f64(w))
        for h in range(H):  # (heads with little memory have much smaller outputs)
            assert normwise(got[b, :, h], want[:, h]) < (1e-5 if dtype == "float32" else 6e-3), (b, h, cuts)
            assert normwise(f64(state[b, h]), end[h]) < (1e-5 if path == 1 or dtype == "float32" else 5e-5)


@pytest.mark.parametrize("dtype,d,dv", [("float32", 8, 24), ("float32", 128, 128), ("float32", 200, 40), ("bfloat16", 24, 40),
                                        ("bfloat16", 128, 128), ("bfloat16", 264, 16)])
def test_decayed_attention_token_by_token(L, dtype, d, dv):
    decayed_case(L, dtype, [1], 1, 2, d, dv, [0.9, 0.5], 1)
    decayed_case(L, dtype, [17, 2, 1, 1, 33], 2, 3, d, dv, [0.999, 0.05, 1.0], 1, seed=1)


@pytest.mark.parametrize("cuts,batch", [([128], 1), ([300], 1), ([127, 2, 1, 129], 1), ([60, 256, 1, 70], 3), ([1, 2, 200], 2)])
def test_decayed_attention_in_chunks(L, cuts, batch):
    decayed_case(L, "bfloat16", cuts, batch, 4, 128, 128, [0.999, 0.6, 1.0, 0.02], 2)
    decayed_case(L, "bfloat16", cuts, batch, 3, 128, 128, [0.97, 0.0, 0.9999], 0, seed=1)


def test_decayed_attention_refuses_chunks_of_other_sizes(L):
    with pytest.raises(ValueError):
        decayed_case(L, "bfloat16", [130], 1, 2, 64, 128, [0.9, 0.9], 2)
    with pytest.raises(ValueError):
        decayed_case(L, "float32", [130], 1, 2, 128, 128, [0.9, 0.9], 2)


def test_a_long_sequence_in_chunks_equals_token_by_token(L):
    """More chunks than the device has multiprocessors, and a value of the first token that only a decay of 1 keeps."""
    rng = np.random.default_rng(2)
    T, H = 3000, 8
    rows = dev(rng.standard_normal((1, T, 3 * H * 128)) * 0.5, torch.bfloat16)
    w = dev(np.float32([1.0, 0.9999, 0.999, 0.99, 0.9, 0.5, 0.1, 0.0]))
    got = []
    for path in (1, 2):
        state, o = torch.zeros(1, H, 128, 128, device="cuda"), torch.empty(1, T, H, 128, dtype=torch.bfloat16, device="cuda")
        for first, last in ((0, 1111), (1111, T)):
            p = rows[:, first:].data_ptr()
            check(L.ytcuda_decayed_attn_fwd(1, p, p + H * 256, p + 2 * H * 256, rows.shape[-1], o[:, first:].data_ptr(),
                                            state.data_ptr(), w.data_ptr(), 1, last - first, H, 128, 128, int(first == 0), path,
                                            stream()))
        got.append((f64(o), f64(state)))
    for h in range(H):
        assert normwise(got[1][0][:, :, h], got[0][0][:, :, h]) < 5e-3
        assert normwise(got[1][1][:, h], got[0][1][:, h]) < 5e-5


# ---------------------------------------------------------------- attention over cached latents
def latent_case(L, dtype, batch, n, pos0, H, d, rot, dv, rank, seed=0):
    """Few rows over a cache; every second row's query points at one position, at and around borders of tiles and slices."""
    rng = np.random.default_rng(seed)
    tt, code = kind(dtype)
    S, cap = pos0 + n, pos0 + n + 5
    uk = dev(rng.standard_normal((H * d, rank)) / np.sqrt(rank), torch.bfloat16)
    uv = dev(rng.standard_normal((H * dv, rank)) / np.sqrt(rank), torch.bfloat16)
    cache = rng.standard_normal((batch, cap, rank + rot))
    cache[:, S:] = 1e4  # rows behind the newest position
    q = rng.standard_normal((batch, n, H, d + rot))
    ukn = f64(uk).reshape(H, d, rank)
    places = [p for p in (0, 1, S - 2, 62, 63, 64, 65, 127, 128, 191, 192) if p >= 0]
    for b in range(batch):
        for t in range(0, n, 2):
            j = min(places[(b + t // 2) % len(places)], pos0 + t)
            for h in range(H):
                q[b, t, h, :d] = 1.5 * ukn[h] @ cache[b, j, :rank]
    qd, cd = dev(q, tt), dev(cache, tt)
    freq = np.power(300.0, -np.arange(rot // 2) * 2.0 / max(rot, 1)).astype(np.float32)
    fd = dev(freq if rot else np.ones(1, np.float32))
    out = torch.empty(batch, n, H, dv, dtype=tt, device="cuda")
    scale = 0.4
    check(L.ytcuda_latent_attn_fwd(code, qd.data_ptr(), uk.data_ptr(), uv.data_ptr(), cd.data_ptr(), cap, out.data_ptr(), batch,
                                   n, pos0, H, d, rot, dv, rank, fd.data_ptr(), scale, stream()))
    qn, cn = f64(qd), f64(cd)
    for b in range(batch):
        c, r = cn[b, :S, :rank], cn[b, :S, None, rank:]
        k = np.concatenate([np.einsum("sr,hdr->shd", c, ukn), np.repeat(r, H, 1)], -1)
        v = np.einsum("sr,hdr->shd", c, f64(uv).reshape(H, dv, rank))
        qq = np.concatenate([qn[b, ..., :d], P.rotate(qn[b, ..., d:], range(pos0, S), 300.0, rot)], -1)
        want = P.causal_attention(qq, k, v, scale)
        assert normwise(f64(out[b]), want) < (2e-5 if dtype == "float32" else 6e-3), (b, n, pos0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,rot,dv,rank", [(3, 24, 16, 40, 48), (17, 64, 32, 64, 128), (1, 128, 64, 128, 512),
                                             (4, 8, 0, 24, 16), (2, 40, 48, 16, 592)])
def test_latent_attention_of_few_rows(L, dtype, H, d, rot, dv, rank):
    for batch, n, pos0 in ((1, 1, 0), (1, 2, 62), (1, 1, 63), (2, 3, 64), (1, 6, 126), (3, 1, 300), (1, 2, 700), (1, 9, 190)):
        latent_case(L, dtype, batch, n, pos0, H, d, rot, dv, rank, seed=pos0)


# ---------------------------------------------------------------- the other mechanisms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,cols", [(40, 48), (2048, 2048), (5000, 5000)])
def test_gated_rows(L, dtype, width, cols):
    rng = np.random.default_rng(width)
    tt, code = kind(dtype)
    x, g = np.zeros((5, cols)), rng.standard_normal((5, cols + 8)) * 3
    x[:, :width] = rng.standard_normal((5, width))
    w = np.zeros(cols, np.float32)
    w[:width] = rng.standard_normal(width)
    xd, gd, wd = dev(x, tt), dev(g, tt), dev(w)
    for norm in (False, True):
        o = torch.empty(5, cols, dtype=tt, device="cuda")
        check(L.ytcuda_gated_rows(code, xd.data_ptr(), cols, gd.data_ptr(), cols + 8, o.data_ptr(), cols, 5, cols, width,
                                  wd.data_ptr() if norm else None, 1e-3, stream()))
        want = f64(xd)
        if norm:
            want[:, :width] = rms_norm(want[:, :width], w[:width].astype(np.float64), 1e-3)
            want[:, width:] = 0
        assert normwise(f64(o), want * P.sigmoid(f64(gd)[:, :cols])) < (1e-6 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_norm_without_a_norm_in_front(L, dtype):
    rng = np.random.default_rng(0)
    tt, code = kind(dtype)
    x, y, w = (dev(rng.standard_normal(s).astype(np.float32)) for s in ((4, 1032), (4, 1032), (1032,)))
    want = f64(x) + rms_norm(f64(y), f64(w), 1e-2)
    h = torch.empty(4, 1032, dtype=tt, device="cuda")
    check(L.ytcuda_residual_norm(x.data_ptr(), y.data_ptr(), w.data_ptr(), None, h.data_ptr(), code, 4, 1032, 1032, 1e-2, stream()))
    assert normwise(f64(x), want) < 1e-6
    assert normwise(f64(h), want) < (1e-6 if dtype == "float32" else 4e-3)
    check(L.ytcuda_residual_norm(x.data_ptr(), None, None, None, h.data_ptr(), code, 4, 1032, 1032, 1e-2, stream()))
    assert normwise(f64(h), want) < (1e-6 if dtype == "float32" else 4e-3) and normwise(f64(x), want) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("m,n,k", [(3, 40, 24), (130, 300, 264), (700, 512, 1024), (300, 46, 72)])
def test_linear_activations(L, dtype, m, n, k):
    rng = np.random.default_rng(m)
    tt, code = kind(dtype)
    x, w = dev(rng.standard_normal((m, k)), tt), dev(rng.standard_normal((n, k)) / np.sqrt(k) * 1.5, torch.bfloat16)
    z = f64(x) @ f64(w).T
    for cols in (0, 17, n - 1):
        want = z.copy()
        want[:, :cols] = silu(z[:, :cols])
        linear_case(L, code, 4, x, w, want, cols, 0.0, dtype)
    linear_case(L, code, 3, x, w, P.squared_relu(z), 0, 0.0, dtype)
    for limit in (0.3, 2.0):
        linear_case(L, code, 5, x, w, P.clamped_gate(z[:, ::2], z[:, 1::2], limit), 0, limit, dtype)


def linear_case(L, code, act, x, w, want, cols, limit, dtype):
    y = torch.empty(want.shape, dtype=x.dtype, device="cuda")
    check(L.ytcuda_linear_act(code, act, x.data_ptr(), x.shape[1], w.data_ptr(), y.data_ptr(), y.shape[1], x.shape[0],
                              w.shape[0], x.shape[1], cols, limit, None, 1, stream()))
    z = np.abs(f64(x)) @ np.abs(f64(w)).T  # (bounded results are small beside the sums they come from)
    tol = max(2e-6 * (1 + limit), 1e-7 * z.max() / np.abs(want).max()) if dtype == "float32" else 5e-3
    assert normwise(f64(y), want) < tol, (act, cols, limit)


@pytest.mark.parametrize("experts,top", [(8, 2), (16, 1), (60, 8), (5, 5), (1, 1), (300, 6)])
def test_sigmoid_router(L, experts, top):
    rng = np.random.default_rng(experts)
    rows = 41
    z = (rng.standard_normal((rows, experts)) * np.linspace(1, 30, rows)[:, None]).astype(np.float32)  # also scores that round to 1
    zd, ch = dev(z), torch.empty(rows, top, dtype=torch.int32, device="cuda")
    rk, w, cnt = torch.empty_like(ch), torch.empty(rows, top, device="cuda"), torch.zeros(experts, dtype=torch.int32, device="cuda")
    check(L.ytcuda_moe_route(zd.data_ptr(), experts, None, rows, experts, 0, top, 1, 1, 1, ch.data_ptr(), w.data_ptr(),
                             rk.data_ptr(), cnt.data_ptr(), stream()))
    for t in range(rows):
        want, ww = P.route(z[t].astype(np.float64), top)
        assert ch[t].tolist() == want and np.abs(w[t].cpu().numpy() - ww).max() < 1e-6
    assert int(cnt.sum()) == rows * top


# ---------------------------------------------------------------- the model
@pytest.fixture(scope="module")
def cases():
    out = {}
    for name, make in Z.CONFIGS.items():
        cfg = make()
        w = Z.weights(cfg, seed=len(name))
        toks = np.random.default_rng(5).integers(0, cfg.vocab, 150).tolist()
        out[name] = (cfg, w, toks, P.forward(cfg.to_dict(), Z.floats(w), toks))
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_prompt_portions_and_decoding(D, cases, name, dtype):
    """The whole prompt in one call, in portions down to two tokens, and token by token: the same logits everywhere, also in
    the first positions; with passes shorter than a call (chunk 32)."""
    cfg, w, toks, want = cases[name]
    whole = None
    for chunk, cuts in ((4096, [len(toks)]), (32, [len(toks)]), (32, [3, 2, 7, 2, 31, 1, 2, 40]), (4096, [2]), (32, [5, 1]),
                        (4096, [1]), (4096, [70, 1, 17, 1, 2])):
        m = model(D, cfg, w, dtype, max_tokens=len(toks), chunk=chunk)
        got = run(m, toks, cuts)
        close(got, want, dtype)
        whole = got if whole is None else whole
        same(got, whole, dtype)
        assert m.get_kv_cache_len() == len(toks)
        m.check_status()
        m.close()


def dense_config(layers, **kw):
    return Z.config(layers, width=72, vocab=110, **kw)


@pytest.mark.parametrize("H,d,rot,dv,rank", [(4, 24, 40, 64, 64), (3, 96, 32, 128, 136), (2, 120, 40, 72, 48), (6, 20, 12, 24, 40)])
def test_bf16_without_a_router(D, H, d, rot, dv, rank):
    """Dense layers in bf16: every position, in every portion, within 4 % - both tile widths of the tensor-core attention,
    padded heads, head dims beyond the tiles, linear attention in chunks and token by token."""
    cfg = dense_config([Z.latent(H, d, rot, dv, rank, 56, ff=96), Z.decayed(H, d, dv, ff=96), Z.decayed(2, 144, 24, ff=64),
                        Z.latent(H, d, rot, dv, rank, 40, ff=96)])
    w = Z.weights(cfg, seed=d, key_gain=1.5)
    toks = np.random.default_rng(6).integers(0, cfg.vocab, 300).tolist()
    want = P.forward(cfg.to_dict(), Z.floats(w), toks)
    for cuts in ([300], [130, 2, 3, 65, 17, 1]):
        m = model(D, cfg, w, "bfloat16", max_tokens=300, chunk=100)
        assert rms_error(run(m, toks, cuts), want) < TOL["bfloat16"]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_decode_kernels_match_the_operator_path(D, L, cases, name, dtype):
    cfg, w, toks, _ = cases[name]
    a, b = (model(D, cfg, w, dtype, max_tokens=len(toks), chunk=32) for _ in range(2))
    b.set_decode_path(1)
    same(run(a, toks, [11, 1]), run(b, toks, [11, 1]), dtype)
    n0 = L.ytcuda_launch_count()
    a.reset_kv_cache()
    a.forward(ids(toks[:1]))
    used = L.ytcuda_launch_count() - n0  # (one more than the step's kernels: the position word)
    assert used <= 2 + sum((3 if x.mixer == D.DECAYED else 6) + (0, 2, 3)[x.mlp] for x in cfg.layers)
    a.close()
    b.close()


def test_long_decoding(D):
    """Hundreds of tokens decoded one by one, with a decay that forgets nothing."""
    cfg = Z.config([Z.decayed(2, 16, 24, decay=[1.0, 0.98], ff=24),
                    Z.latent(2, 8, 8, 24, 24, 16, mlp="moe", ff=16, experts=4, top=2, limit=1.0, shared_ff=8, shared_limit=1.0)],
                   width=32, vocab=40)
    w = Z.weights(cfg, seed=3)
    toks = np.random.default_rng(1).integers(0, cfg.vocab, 520).tolist()
    want = P.forward(cfg.to_dict(), Z.floats(w), toks)
    m = model(D, cfg, w, "float32", max_tokens=1000)
    close(run(m, toks, [50, 1]), want, "float32")
    m.close()


def lookup_weights(cfg):
    """One layer over one-hot tokens: token 2 asks for token 1 (token 3 fills), and its logits 1 and 3 tell whether it saw it."""
    f = {n: np.zeros(s, np.float32) for n, s in cfg.tensor_shapes().items()}
    for n in f:
        if "norm" in n:
            f[n][:] = 1
    f["embed"][np.arange(cfg.vocab), np.arange(cfg.vocab)] = 1
    f["head"][1, 9] = f["head"][3, 10] = 3
    m = "l0.mix."
    f[m + "o"][9, 1] = f[m + "o"][10, 2] = 1
    if cfg.layers[0].mixer == 1:
        f[m + "dq"][0, 2] = f[m + "dkv"][0, 1] = f[m + "dkv"][1, 3] = 1
        f[m + "uq"][0, 0] = 4             # token 2 asks along dimension 0 ...
        f[m + "uk"][0, 0] = 1             # ... token 1 answers
        f[m + "uv"][1, 0] = f[m + "uv"][2, 1] = 1
    else:
        big = 12                          # (silu(big) is big)
        f[m + "q"][0, 2] = f[m + "k"][0, 1] = f[m + "v"][1, 1] = big
        f[m + "q"][1, 2] = f[m + "k"][1, 3] = 1e-2
        f[m + "v"][2, 3] = big
    return {n: Z.f32_to_bf16_bits(a) for n, a in f.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layer", [Z.latent(1, 8, 4, 8, 8, 8, scale=1.0, mlp=None),
                                   Z.decayed(1, 8, 8, decay=[1.0], mlp=None)])
def test_one_far_token_among_hundreds_is_found(D, dtype, layer):
    cfg = Z.config([layer], width=16, vocab=8, scale=1.0)
    w = lookup_weights(cfg)
    m = model(D, cfg, w, dtype, max_tokens=900, chunk=128)
    for at in (0, 1, 62, 63, 64, 127, 128, 255):
        for gap in (1, 2, 64, 127, 129, 400):
            toks = [3] * at + [1] + [3] * (gap - 1) + [2]
            plain = P.forward(cfg.to_dict(), Z.floats(w), toks)[-1]
            without = P.forward(cfg.to_dict(), Z.floats(w), [3 if t == 1 else t for t in toks])[-1] if at + gap < 140 else None
            assert plain[1] > plain[3] and (without is None or without[1] < without[3] + 1e-6)
            for cuts in ([len(toks)], [len(toks) - 1, 1], [max(1, len(toks) - 2), 2], [max(1, len(toks) - 60), 60]):
                m.reset_kv_cache()
                assert rms_error(run(m, toks, cuts)[-1][None], plain[None]) < (1e-4 if dtype == "float32" else 2e-2)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_caches_and_states_that_are_used_again_leave_no_trace(D, cases, dtype):
    cfg, w, toks, _ = cases["mixed"]
    other = np.random.default_rng(9).integers(0, cfg.vocab, 75).tolist()
    m = model(D, cfg, w, dtype, max_tokens=len(toks), chunk=32)
    for cuts in ([9, 1, 23, 1], [1], [60, 2]):
        m.reset_kv_cache()
        first = run(m, toks[:60], cuts)
        for between in ([75], [1]):
            m.reset_kv_cache()
            assert m.get_kv_cache_len() == 0
            run(m, other, between)
            m.reset_kv_cache()
            assert np.array_equal(first, run(m, toks[:60], cuts))
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_batch_equals_each_sequence_alone(D, cases, dtype):
    cfg, w, _, _ = cases["mixed"]
    rng = np.random.default_rng(2)
    toks = rng.integers(0, cfg.vocab, (3, 75)).astype(np.int32)
    b = model(D, cfg, w, dtype, batch=3, max_tokens=75, chunk=32)
    got = [b.forward(dev(toks[:, :50])).cpu().numpy()] + [b.forward(dev(toks[:, t:t + 1])).cpu().numpy() for t in range(50, 70)]
    got.append(b.forward(dev(toks[:, 70:])).cpu().numpy())
    b.close()
    m = model(D, cfg, w, dtype, max_tokens=75)
    for s in range(3):
        m.reset_kv_cache()
        alone = run(m, toks[s].tolist(), [50, 1])
        same(np.stack([g[s] for g in got]), np.concatenate([alone[49:70], alone[74:]]), dtype)
    m.close()


@pytest.mark.parametrize("name", list(Z.CONFIGS))
def test_greedy_generation(D, cases, name):
    cfg, w, toks, _ = cases[name]
    prompt = toks[:13]
    want = P.greedy(cfg.to_dict(), Z.floats(w), prompt, 16)
    m = model(D, cfg, w, "float32", max_tokens=64)
    assert m.generate_greedy(ids(prompt), 16).cpu().numpy()[0].tolist() == want
    m.reset_kv_cache()
    assert m.generate_topk(ids(prompt), 16, k=1).cpu().numpy()[0].tolist() == want  # k = 1 is greedy decoding
    m.reset_kv_cache()
    a = m.generate_topk(ids(prompt), 12, k=5, seed=3).cpu().numpy()
    m.reset_kv_cache()
    assert np.array_equal(a, m.generate_topk(ids(prompt), 12, k=5, seed=3).cpu().numpy())
    m.close()


def test_registry_command_line_and_trace(D, cases, tmp_path):
    from ytensor_b200.registry import load_model
    from ytensor_b200.safetensors import write_safetensors
    cfg, w, toks, want = cases["odd"]
    folder = tmp_path / "m"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg.to_dict()))
    write_safetensors(folder / "model.safetensors", w)
    m = load_model(folder, dtype="float32", max_tokens=64)
    assert isinstance(m, D.DerupelForCausalLM)
    greedy = m.generate_greedy(ids(toks[:9]), 8).cpu().numpy()[0].tolist()
    m.close()
    env = dict(os.environ, PYTHONPATH=str(ROOT))
    r = subprocess.run([sys.executable, "-m", "ytensor_b200", "generate", "--model", str(folder), "--dtype", "float32",
                        "--tokens", ",".join(map(str, toks[:9])), "--steps", "8"], capture_output=True, text=True, env=env,
                       timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()[-1].split(",")] == greedy
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:20], "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[20:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[21:23], "want": [1]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}], "end": []}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
                        str(tmp_path), "--max-tokens", "40"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    for step, places in ((0, [19, 3]), (2, [22]), (3, [0])):
        close(np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(-1, cfg.vocab), want[places], "float32")
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
        D.DerupelForCausalLM(Z.config([Z.latent(2, 260, 12)]))
    with pytest.raises(ValueError):
        D.DerupelForCausalLM(cfg, dtype="float16")
    with pytest.raises(ValueError):
        model(D, cfg, dict(w, head=w["head"][:-1]))
