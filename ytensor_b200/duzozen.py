"""Host side of the Duzozen language model: configuration, weights (padding, fusing, upload) and the wrapper over the
model handle of the C ABI (ytcuda_duzozen_*).

The kernels want widths in multiples of 8 and, for the tensor-core attention, head dims of 64 or 128. Any other size is
padded here with zero weights: padded channels of the residual stream, of a head or of a feed-forward stay zero, and
norms run over the true width. torch is used for device memory only."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np

from . import _lib
from ._lib import check, lib
from .causal_lm import CausalLM

MLP_NONE, MLP_DENSE, MLP_MOE = 0, 1, 2


class _ConfigC(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("width", "norm_width", "vocab", "layers", "batch", "max_tokens", "chunk", "dtype")] + \
               [("eps", C.c_float)]


class _LayerC(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("heads", "kv_heads", "dim", "vdim", "window", "v_mix", "mlp", "ff", "experts",
                                       "identity", "top", "groups", "keep")] + \
               [("scale", C.c_float), ("softcap", C.c_float)]


@dataclass
class DuzozenLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float = 0.0     # 0: scores are not capped
    window: int = 0          # 0: every earlier position is visible
    v_mix: bool = False
    mlp: int = MLP_NONE
    ff: int = 0              # dense width, or the width of one expert
    experts: int = 0
    identity: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1

    @staticmethod
    def from_dict(d: dict) -> "DuzozenLayer":
        if d["type"] != "attention":
            raise ValueError(f"unknown mixer '{d['type']}'")
        m = d["mixer"]
        L = DuzozenLayer(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                         scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                         window=int((m.get("mask") or {}).get("size") or 0), v_mix=bool(m.get("v_mix")))
        f = d.get("mlp")
        if f is None:
            return L
        if f["kind"] == "dense":
            L.mlp, L.ff = MLP_DENSE, int(f["ff"])
        elif f["kind"] == "moe":
            r = f["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            L.mlp, L.ff = MLP_MOE, int(f["expert"]["ff"])
            L.experts, L.identity, L.top = int(r["experts"]), int(r.get("identity") or 0), int(r["top"])
            L.groups, L.keep = int(g["count"]), int(g["keep"])
        else:
            raise ValueError(f"unknown feed-forward '{f['kind']}'")
        return L

    def to_dict(self) -> dict:
        m = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "v_mix": self.v_mix}
        if self.softcap:
            m["softcap"] = self.softcap
        if self.window:
            m["mask"] = {"size": self.window}
        f = None
        if self.mlp == MLP_DENSE:
            f = {"kind": "dense", "ff": self.ff}
        elif self.mlp == MLP_MOE:
            f = {"kind": "moe", "expert": {"ff": self.ff},
                 "router": {"experts": self.experts, "identity": self.identity, "top": self.top,
                            "groups": {"count": self.groups, "keep": self.keep}}}
        return {"type": "attention", "mixer": m, "mlp": f}


@dataclass
class DuzozenConfig:
    width: int
    vocab: int
    eps: float
    layers: list = field(default_factory=list)

    @staticmethod
    def from_dict(d: dict) -> "DuzozenConfig":
        return DuzozenConfig(width=int(d["width"]), vocab=int(d["vocab"]), eps=float(d["norm"]["eps"]),
                             layers=[DuzozenLayer.from_dict(x) for x in d["layers"]])

    def to_dict(self) -> dict:
        return {"architecture": "Duzozen", "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                "layers": [x.to_dict() for x in self.layers]}

    def tensor_shapes(self) -> dict:
        """Checkpoint tensor names and shapes."""
        W, s = self.width, {"embed": (self.vocab, self.width)}
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if L.mlp != MLP_NONE else ()):
                s[p + n] = (W,)
            s[p + "mix.q"] = (L.heads * L.dim, W)
            s[p + "mix.k"] = (L.kv_heads * L.dim, W)
            s[p + "mix.v"] = (L.kv_heads * L.vdim, W)
            if L.v_mix:
                s[p + "mix.vmix"] = ()
            s[p + "mix.o"] = (W, L.heads * L.vdim)
            if L.mlp == MLP_DENSE:
                s[p + "mlp.up"], s[p + "mlp.down"] = (L.ff, W), (W, L.ff)
            elif L.mlp == MLP_MOE:
                for e in range(L.experts):
                    s[f"{p}mlp.e{e}.gate"], s[f"{p}mlp.e{e}.up"], s[f"{p}mlp.e{e}.down"] = (L.ff, W), (L.ff, W), (W, L.ff)
                s[p + "mlp.router"] = (L.experts + L.identity, W)
                s[p + "mlp.correction"] = (L.experts + L.identity,)
        s["final.norm"], s["head"] = (W,), (self.vocab, W)
        return s


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


class DuzozenForCausalLM(CausalLM):
    """Device model for `batch` sequences of up to `max_tokens` tokens. dtype "bfloat16": bf16 activations, cache and
    tensor-core products, fp32 residual stream, norms, scores and router; "float32": everything fp32 (weights stay in
    their bf16 storage, the products are the same numbers). chunk: most tokens per sequence that run through the layers
    at once; with it a layer's window bounds its K/V ring."""

    def __init__(self, cfg: DuzozenConfig, batch: int = 1, max_tokens: int = 4096, dtype: str = "bfloat16",
                 chunk: int = 4096):
        import torch
        self.torch = torch
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype must be bfloat16 or float32, not {dtype}")
        self.cfg, self.batch, self.dtype, self.max_tokens = cfg, batch, dtype, max_tokens
        self.L = lib()
        self.width_p = _up8(cfg.width)
        dt = _lib.BF16 if dtype == "bfloat16" else _lib.F32
        cc = _ConfigC(self.width_p, cfg.width, cfg.vocab, len(cfg.layers), batch, max_tokens, chunk, dt, cfg.eps)
        lc = (_LayerC * len(cfg.layers))()
        self.head_dims = []
        for i, x in enumerate(cfg.layers):
            d, dv = self._pad_head(x.dim, x.vdim)
            self.head_dims.append((d, dv))
            lc[i] = _LayerC(x.heads, x.kv_heads, d, dv, x.window, int(x.v_mix), x.mlp, _up8(x.ff), x.experts, x.identity,
                            x.top, x.groups, x.keep, x.scale, x.softcap)
        mixing = [x.kv_heads * 1000003 + x.vdim for x in cfg.layers if x.v_mix]
        if len(set(mixing)) > 1:
            raise ValueError("layers that mix values must have the same kv_heads and vdim")
        h = self.L.ytcuda_duzozen_create(C.byref(cc), C.cast(lc, C.c_void_p))
        if not h:
            raise _lib.YtCudaInvalidArgument(_lib.INVALID_ARG, _lib.last_error())
        self.h = C.c_void_p(h)
        self._keep = []

    def _pad_head(self, dim: int, vdim: int):
        if self.dtype == "bfloat16":
            for size in (64, 128):  # what the tensor-core attention takes
                if max(dim, vdim) <= size:
                    return size, size
        return _up8(dim), _up8(vdim)

    # ---- weights
    def load_weights(self, weights) -> None:
        """weights: checkpoint name -> numpy array (uint16: bf16 bits, or float32) or torch tensor; anything with
        __getitem__ (a dict, a SafetensorsFile)."""
        torch = self.torch
        dev = torch.device("cuda", torch.cuda.current_device())
        pad = torch.nn.functional.pad
        cfg, wp = self.cfg, self.width_p
        shapes = cfg.tensor_shapes()

        def get(name, dtype):
            a = weights[name]
            if not isinstance(a, torch.Tensor):
                a = np.array(a)  # (an own, writable copy)
                a = torch.from_numpy(a.view(np.int16)).view(torch.bfloat16) if a.dtype == np.uint16 else torch.from_numpy(a)
            if tuple(a.shape) != shapes[name]:
                raise ValueError(f"{name}: shape {tuple(a.shape)} does not fit the configuration ({shapes[name]})")
            return a.to(dev).to(dtype)

        def mat(name, rows=0, cols=0):  # zero-padded to rows x cols (0: as it is)
            a = get(name, torch.bfloat16)
            return pad(a, (0, max(0, cols - a.shape[1]), 0, max(0, rows - a.shape[0])))

        def vec(name, size=0):
            a = get(name, torch.float32).reshape(-1)
            return pad(a, (0, max(0, size - a.shape[0])))

        def heads_in(name, n, d, dp):   # [n * d, width] -> [n * dp, width_p]
            a = get(name, torch.bfloat16).reshape(n, d, cfg.width)
            return pad(a, (0, wp - cfg.width, 0, dp - d)).reshape(n * dp, wp)

        def put(name, layer, t):
            t = t.contiguous()
            self._keep.append(t)
            check(self.L.ytcuda_duzozen_set_weight(self.h, name.encode(), layer, t.data_ptr()))

        put("embed", 0, mat("embed", cols=wp))
        put("head", 0, mat("head", cols=wp))
        put("norm", 0, vec("final.norm", wp))
        for i, x in enumerate(cfg.layers):
            p = f"l{i}."
            dp, dvp = self.head_dims[i]
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if x.mlp != MLP_NONE else ()):
                put(n, i, vec(p + n, wp))
            put("qkv", i, torch.cat([heads_in(p + "mix.q", x.heads, x.dim, dp), heads_in(p + "mix.k", x.kv_heads, x.dim, dp),
                                     heads_in(p + "mix.v", x.kv_heads, x.vdim, dvp)]))
            o = get(p + "mix.o", torch.bfloat16).reshape(cfg.width, x.heads, x.vdim)
            put("o", i, pad(o, (0, dvp - x.vdim, 0, 0, 0, wp - cfg.width)).reshape(wp, x.heads * dvp))
            if x.v_mix:
                put("vmix", i, vec(p + "mix.vmix"))
            fp = _up8(x.ff)
            if x.mlp == MLP_DENSE:
                put("up", i, mat(p + "mlp.up", fp, wp))
                put("down", i, mat(p + "mlp.down", wp, fp))
            elif x.mlp == MLP_MOE:
                put("router", i, mat(p + "mlp.router", cols=wp))
                put("correction", i, vec(p + "mlp.correction"))
                if x.experts:
                    gate_up = torch.zeros(x.experts, fp, 2, wp, dtype=torch.bfloat16, device=dev)
                    down = torch.zeros(x.experts, wp, fp, dtype=torch.bfloat16, device=dev)
                    for e in range(x.experts):
                        q = f"{p}mlp.e{e}."
                        gate_up[e, :, 0] = mat(q + "gate", fp, wp)
                        gate_up[e, :, 1] = mat(q + "up", fp, wp)
                        down[e] = mat(q + "down", wp, fp)
                    put("up", i, gate_up)
                    put("down", i, down)

    # ---- sequences
    def reset_kv_cache(self) -> None:
        check(self.L.ytcuda_duzozen_reset(self.h))

    def get_kv_cache_len(self) -> int:
        return self.L.ytcuda_duzozen_cache_len(self.h)

    def set_decode_path(self, path: int) -> None:
        """One new token of a single sequence: 0 the CUDA graph of fused decode kernels, 1 one launch per operator."""
        check(self.L.ytcuda_duzozen_set_decode_path(self.h, int(path)))

    def forward_rows(self, ids, want):
        """ids int32 [batch, len] (device) -> logits fp32 [len(want), vocab] of rows `want` of the flattened input."""
        torch = self.torch
        assert ids.is_cuda and ids.dtype == torch.int32 and ids.shape[0] == self.batch and ids.is_contiguous()
        logits = torch.empty(len(want), self.cfg.vocab, dtype=torch.float32, device=ids.device)
        rows = (C.c_int32 * len(want))(*want)
        check(self.L.ytcuda_duzozen_forward(self.h, ids.data_ptr(), ids.shape[1], C.cast(rows, C.c_void_p), len(want),
                                            logits.data_ptr(), torch.cuda.current_stream().cuda_stream))
        return logits

    def forward(self, ids):
        n = ids.shape[1]
        return self.forward_rows(ids, [b * n + n - 1 for b in range(self.batch)])

    def forward_at(self, ids, want):
        return self.forward_rows(ids, list(want))

    def close(self) -> None:
        if getattr(self, "h", None):
            self.L.ytcuda_duzozen_destroy(self.h)
            self.h = None
            self._keep = []

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass
