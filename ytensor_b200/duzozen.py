"""Host side of the Duzozen language model: configuration and weights (padding, fusing) for the model handle of the C ABI
(ytcuda_duzozen_*; native_lm.py has what it shares with other models).

The kernels want widths in multiples of 8 and, for the tensor-core attention, head dims of 64 or 128. Any other size is
padded here with zero weights: padded channels of the residual stream, of a head or of a feed-forward stay zero, and
norms run over the true width."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

from .native_lm import MLP_DENSE, MLP_MOE, MLP_NONE, NativeLM, up8


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


class DuzozenForCausalLM(NativeLM):
    """With `chunk`, a layer's window bounds its K/V ring."""

    native = "duzozen"

    def _create(self, chunk, dtype):
        cfg = self.cfg
        cc = _ConfigC(self.width_p, cfg.width, cfg.vocab, len(cfg.layers), self.batch, self.max_tokens, chunk, dtype, cfg.eps)
        lc = (_LayerC * len(cfg.layers))()
        self.head_dims = []
        for i, x in enumerate(cfg.layers):
            d, dv = self._pad_head(x.dim, x.vdim)
            self.head_dims.append((d, dv))
            lc[i] = _LayerC(x.heads, x.kv_heads, d, dv, x.window, int(x.v_mix), x.mlp, up8(x.ff), x.experts, x.identity,
                            x.top, x.groups, x.keep, x.scale, x.softcap)
        mixing = [x.kv_heads * 1000003 + x.vdim for x in cfg.layers if x.v_mix]
        if len(set(mixing)) > 1:
            raise ValueError("layers that mix values must have the same kv_heads and vdim")
        return cc, lc

    def _pad_head(self, dim: int, vdim: int):
        if self.dtype == "bfloat16":
            for size in (64, 128):  # what the tensor-core attention takes
                if max(dim, vdim) <= size:
                    return size, size
        return up8(dim), up8(vdim)

    def _load(self, ck):
        cfg, wp, put = self.cfg, self.width_p, self._put
        for i, x in enumerate(cfg.layers):
            p = f"l{i}."
            dp, dvp = self.head_dims[i]
            for n in ("norm1", "norm1b") + (("norm2", "norm2b") if x.mlp != MLP_NONE else ()):
                put(n, i, ck.vec(p + n, wp))
            put("qkv", i, self.torch.cat([ck.heads_out(p + "mix.q", x.heads, x.dim, dp, wp),
                                          ck.heads_out(p + "mix.k", x.kv_heads, x.dim, dp, wp),
                                          ck.heads_out(p + "mix.v", x.kv_heads, x.vdim, dvp, wp)]))
            put("o", i, ck.heads_in(p + "mix.o", x.heads, x.vdim, dvp, wp))
            if x.v_mix:
                put("vmix", i, ck.vec(p + "mix.vmix"))
            fp = up8(x.ff)
            if x.mlp == MLP_DENSE:
                put("up", i, ck.mat(p + "mlp.up", fp, wp))
                put("down", i, ck.mat(p + "mlp.down", wp, fp))
            elif x.mlp == MLP_MOE:
                put("router", i, ck.mat(p + "mlp.router", cols=wp))
                put("correction", i, ck.vec(p + "mlp.correction"))
                if x.experts:
                    up, down = ck.experts(p + "mlp.", x.experts, fp, wp)
                    put("up", i, up)
                    put("down", i, down)
