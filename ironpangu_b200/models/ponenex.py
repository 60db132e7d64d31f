"""Ponenex: a decoder of latent-attention layers with routed experts, a norm before AND after every sublayer (gains stored as their
distance from one) and a scaled residual update over an f32 residual stream.

  h = rms(x) (1 + w1);  x += mult * rms(mixer(h)) (1 + w1b);  the same around the feed-forward with w2 / w2b
  latent_attention   queries and keys / values through latents (rms with plain gains); per head an unrotated part against W_uk c and a
                     rotated part (half layout) against one key part shared by all heads; softmax of scores * scale over the last
                     ``mask.size`` positions; head h times sigmoid(W_g h)_h; W_o. Pages hold the latent and the rotated key part
  moe                router logits + bias, the largest ``top`` chosen, softmax over just these; SwiGLU experts; a shared expert times
                     sigmoid(W_sg h)

``PonenexDecoder`` and ``PonenexRows`` are the decode and packed-step executors (``stream_decoder.py``); the mechanisms are
``ops/latent_attn.py`` and ``ops/routed_experts.py``. In bf16 the linears take bf16 operands with f32 accumulation; norms, rotations,
scores, weights, the router and the residual are f32. With ``dtype=torch.float32`` every product is a true f32 FMA.

A checkpoint directory is ``config.json`` (``"architecture": "Ponenex"``) + safetensors; see :func:`weight_shapes` for the names."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import stream_norm as N
from ..ops.latent_attn import LatentBuffers, LatentMixer, LatentShape
from ..ops.linear_attn import DevicePlan, RotaryTables
from ..ops.routed_experts import ExpertBuffers, ExpertsShape, RoutedExperts
from ..parallel.fabric import Fabric
from . import checkpoint
from .checkpoint import pad8
from .stream_decoder import ATTN_ROWS, BF16, F32, StreamDecoder, StreamRows

KERNEL_UNITS = ("misc", "post_norm", "linear_f32", "latent_attn", "tc_heads", "moe_rows", "moe_prefill", "tc_grouped", "decode_post_norm", "window_attn",
                "fa_prefill", "decode_moe", "sampling", "tc_gemm", "tc_gemm_2sm")


# ---------------------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------------------
@dataclass
class LayerConfig:
    mixer: LatentShape
    mlp: Optional[ExpertsShape] = None       # None: no feed-forward


@dataclass
class PonenexConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float = 1.0
    embed_scale: float = 1.0
    layers: List[LayerConfig] = field(default_factory=list)
    page_tokens: int = 16

    @staticmethod
    def from_dict(j: dict) -> "PonenexConfig":
        if j.get("architecture") != "Ponenex":
            raise ValueError(f"not a Ponenex configuration (architecture {j.get('architecture')!r})")
        width, layers = int(j["width"]), []
        for i, e in enumerate(j["layers"]):
            m, f = e["mixer"], e.get("mlp")
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            rot = m.get("rot") or {}
            mixer = LatentShape(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                q_rank=int(m["q_rank"]), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
                                window=int((m.get("mask") or {}).get("size", 0)), scale=float(m["scale"]))
            mlp = None
            if f is not None:
                if f.get("kind") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
                mlp = ExpertsShape(width, int(f["router"]["experts"]), int(f["router"]["top"]), int(f["expert"]["ff"]), int((f.get("shared") or {}).get("ff", 0)))
            layers.append(LayerConfig(mixer, mlp))
        return PonenexConfig(int(j["vocab"]), width, float(j["norm"]["eps"]), float(j.get("residual_mult", 1.0)), float((j.get("embedding") or {}).get("scale", 1.0)),
                             layers).validate()

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m, f = l.mixer, l.mlp
            d = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale,
                 "mask": {"size": m.window}, "rot": {"dims": m.rot_dims, "base": m.rot_base}}
            g = None
            if f is not None:
                g = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff:
                    g["shared"] = {"ff": f.shared_ff}
            out.append({"type": "latent_attention", "mixer": d, "mlp": g})
        return {"architecture": "Ponenex", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "residual_mult": self.residual_mult,
                "embedding": {"scale": self.embed_scale}, "layers": out}

    def validate(self) -> "PonenexConfig":
        if not self.layers:
            raise ValueError("no layers")
        for i, l in enumerate(self.layers):
            try:
                l.mixer.check()
                if l.mlp is not None:
                    l.mlp.check()
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
        return self

    @property
    def window(self) -> int:
        """The longest window when every layer has one, else 0."""
        w = [l.mixer.window for l in self.layers]
        return max(w) if all(w) else 0

    def param_count(self) -> int:
        return checkpoint.param_count(weight_shapes(self))

    def active_params(self) -> int:
        """Parameters a token uses: all but the experts it does not choose, and one row of the embedding."""
        idle = sum((l.mlp.experts - l.mlp.top) * 3 * l.mlp.ff * self.width for l in self.layers if l.mlp)
        return self.param_count() - idle - (self.vocab - 1) * self.width

    @staticmethod
    def tiny() -> "PonenexConfig":
        """Layers of different sizes, one without a shared expert, one without a feed-forward; odd sizes."""
        a = LatentShape(6, 40, 24, 56, 72, 48, 24, 1e4, 24, 0.13)
        b = LatentShape(3, 20, 16, 24, 104, 36, 12, 5e5, 50, 0.17)
        return PonenexConfig(384, 136, 1e-5, 0.6, 1.7, [LayerConfig(a, ExpertsShape(136, 6, 2, 40, 72)), LayerConfig(b, None),
                                                        LayerConfig(b, ExpertsShape(136, 5, 3, 36)), LayerConfig(a, ExpertsShape(136, 6, 1, 40, 24))]).validate()

    @staticmethod
    def text(layers: int = 16, width: int = 2048, heads: int = 16, dim: int = 128, rot_dim: int = 64, vdim: int = 128, kv_rank: int = 512, q_rank: int = 768,
             experts: int = 64, top: int = 8, ff: int = 768, shared_ff: int = 768, vocab: int = 128000, window: int = 1024) -> "PonenexConfig":
        """A stack of equal layers; the defaults are a small mixture model (5.6 B parameters, 1.2 B of them active)."""
        m = LatentShape(heads, dim, rot_dim, vdim, kv_rank, q_rank, rot_dim, 1e6, window, (dim + rot_dim) ** -0.5)
        return PonenexConfig(vocab, width, 1e-5, 0.5, 1.0, [LayerConfig(m, ExpertsShape(width, experts, top, ff, shared_ff)) for _ in range(layers)]).validate()


PRESETS = {"ponenex-tiny": PonenexConfig.tiny, "ponenex-text": PonenexConfig.text}


# ---------------------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------------------
def weight_shapes(c: PonenexConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names -> shapes (bf16 in the file)."""
    s = {"embed": (c.vocab, c.width), "final.norm": (c.width,), "head": (c.vocab, c.width)}
    for i, l in enumerate(c.layers):
        p, m, f = f"l{i}.", l.mixer, l.mlp
        s.update({p + "norm1": (c.width,), p + "norm1b": (c.width,),
                  p + "mix.dq": (m.q_rank, c.width), p + "mix.dq.norm": (m.q_rank,), p + "mix.uq": (m.heads * (m.dim + m.rot_dim), m.q_rank),
                  p + "mix.dkv": (m.kv_rank + m.rot_dim, c.width), p + "mix.dkv.norm": (m.kv_rank,), p + "mix.uk": (m.heads * m.dim, m.kv_rank),
                  p + "mix.uv": (m.heads * m.vdim, m.kv_rank), p + "mix.g": (m.heads, c.width), p + "mix.o": (c.width, m.heads * m.vdim)})
        if f is None:
            continue
        s.update({p + "norm2": (c.width,), p + "norm2b": (c.width,), p + "mlp.router": (f.experts, c.width), p + "mlp.router.b": (f.experts,)})
        units = [(f"e{e}.", f.ff) for e in range(f.experts)] + ([("shared.", f.shared_ff)] if f.shared_ff else [])
        for name, ff in units:
            q = p + "mlp." + name
            s.update({q + "gate": (ff, c.width), q + "up": (ff, c.width), q + "down": (c.width, ff)})
        if f.shared_ff:
            s[p + "mlp.shared.sg"] = (1, c.width)
    return s


def random_weights(c: PonenexConfig, device, seed: int = 0, std: float = 0.02) -> Dict[str, torch.Tensor]:
    """Random-init checkpoint tensors: N(0, std) matrices, centred gains N(0, std), the latents' plain gains 1 + N(0, std)."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        t = torch.empty(shape, dtype=BF16, device=device).normal_(0.0, std, generator=g)
        out[name] = t + 1.0 if name.endswith(("dq.norm", "dkv.norm")) else t
    return out


def save_checkpoint(path, c: PonenexConfig, weights: Dict[str, torch.Tensor]) -> None:
    checkpoint.save(path, c, weights)


def load_checkpoint(path) -> tuple:
    """``(config, weights on the host)`` of a checkpoint directory; every expected tensor must be there with its shape."""
    return checkpoint.load(path, PonenexConfig.from_dict, weight_shapes)


# ---------------------------------------------------------------------------------------------------------------------------
# executors
# ---------------------------------------------------------------------------------------------------------------------------
class _Rows:
    """Step buffers for up to ``rows`` rows (leading dimensions padded to 8 elements, padding zero)."""

    def __init__(self, dec: "PonenexDecoder", rows: int, chunked: bool):
        c, dev, A = dec.cfg, dec.fabric.device, dec.dtype
        z = lambda n, dt=A: torch.zeros(rows, pad8(n), dtype=dt, device=dev)
        self.rows = rows
        self.x, self.x2 = z(c.width, F32), z(c.width, F32)           # residual stream (two: fused prologues write the other one)
        self.xa, self.y = z(c.width), z(c.width, F32)
        shapes = [l.mixer for l in c.layers]
        self.latent = LatentBuffers(shapes, rows, A, dev, chunked=chunked, max_context=dec.max_context, group=ATTN_ROWS)
        mlps = [l.mlp for l in c.layers if l.mlp is not None]
        self.experts = ExpertBuffers(mlps, rows, A, dev) if mlps else None
        self.rotary = RotaryTables([(m.rot_dims, m.rot_base) for m in shapes], rows, dev)


class PonenexDecoder(StreamDecoder):
    """Decode executor: see :class:`StreamDecoder`."""

    name = "ponenex"

    def make_rows(self, rows: int, chunked: bool) -> _Rows:
        return _Rows(self, rows, chunked)

    def _load(self, W: Dict[str, torch.Tensor]) -> None:
        c, dev = self.cfg, self.fabric.device
        self.embed, self.head = self._mat(W, "embed"), self._mat(W, "head")
        gain = lambda n: 1.0 + self._vec(W, n)
        out_gain = lambda n: c.residual_mult * (1.0 + self._vec(W, n))          # the residual factor belongs to the output norm
        self.final_norm = gain("final.norm")
        self.layers: List[dict] = []
        for i, l in enumerate(c.layers):
            p = f"l{i}."
            L = {"mix": LatentMixer(l.mixer, W, p + "mix.", dev, self.dtype, max_context=self.max_context), "norm1": gain(p + "norm1"), "norm1b": out_gain(p + "norm1b"),
                 "ff": None}
            if l.mlp is not None:
                L.update(ff=RoutedExperts(l.mlp, W, p + "mlp.", dev, self.dtype), norm2=gain(p + "norm2"), norm2b=out_gain(p + "norm2b"))
            self.layers.append(L)
        # the fused decode chain streams unpadded operands
        self.fused = self.dtype == BF16 and c.width % 8 == 0 and all(n % 8 == 0 for l in c.layers for n in (l.mixer.q_rank, l.mixer.heads * l.mixer.vdim))

    def _state_bytes(self) -> tuple:
        es = torch.empty((), dtype=self.dtype).element_size()
        return sum(l.mixer.row for l in self.cfg.layers) * es, 0

    def _make_states(self) -> None:
        for L in self.layers:
            L["mix"].make_pages(self.num_pages, self.cfg.page_tokens)

    @classmethod
    def from_checkpoint(cls, path, fabric: Fabric, **kw) -> "PonenexDecoder":
        c, w = load_checkpoint(path)
        return cls(c, w, fabric, **kw)

    # -- layers ------------------------------------------------------------------------------------------------------------
    def _next_gain(self, i: int, final: bool) -> Optional[torch.Tensor]:
        """Gain of the norm that follows layer ``i``'s last residual update (None: nothing reads the operand)."""
        return self.layers[i + 1]["norm1"] if i + 1 < len(self.layers) else self.final_norm if final else None

    def _layers(self, B: _Rows, m: int, tok, pos, slot, plan: Optional[DevicePlan], final: bool, probe: Optional[list] = None) -> None:
        """All layers over ``m`` rows as separate row operators and matrix products; the residual ends in ``B.x``, and with ``final`` the
        normalised rows for the output matrix in ``B.xa``."""
        c, st, W = self.cfg, self.fabric.desc.status, self.cfg.width
        x, xa, y, lat = B.x[:m, :W], B.xa[:m], B.y[:m, :W], B.latent
        N.embed_rows(tok, self.embed, x, xa, scale=c.embed_scale, gain=self.layers[0]["norm1"], eps=c.eps, status_ptr=st)
        B.rotary.fill(pos)
        if B.experts is not None:
            B.experts.start(m)
        for i, L in enumerate(self.layers):
            mix, ff, after = L["mix"], L["ff"], self._next_gain(i, final)
            s = mix.shape
            N.linear(xa, mix.w_in, lat.proj[:m, :s.in_cols], status_ptr=st)
            mix.mix(lat, m, B.rotary.get(s.rot_dims, s.rot_base), pos, slot, plan, self.page_table, c.eps, st)
            N.linear(lat.mixed[s.heads * s.vdim][:m], mix.w_o, y, status_ptr=st)
            N.post_norm_add(y, L["norm1b"], c.eps, x, xa, after if ff is None else L["norm2"])
            if ff is not None:
                ff.rows(B.experts, m, xa, L["norm2b"], after, c.eps, B.x[:m], st)
            if probe is not None:
                probe.append(x.clone())

    def _layers_fused(self, B: _Rows, n: int, tok, pos, slot) -> None:
        """Decode rows: every norm and residual update inside the linear that follows it. Ends like :meth:`_layers` with ``final``."""
        c, st = self.cfg, self.fabric.desc.status
        x, x2, xa, y, lat = B.x[:n], B.x2[:n], B.xa[:n], B.y[:n], B.latent
        N.embed_rows(tok, self.embed, x, xa, scale=c.embed_scale, gain=self.layers[0]["norm1"], eps=c.eps, status_ptr=st)
        B.rotary.fill(pos)
        owed = None                            # gain of the sublayer output in y that the residual still lacks
        for L in self.layers:
            mix, ff = L["mix"], L["ff"]
            s = mix.shape
            proj = lat.proj[:n, :s.in_cols]
            if owed is None:
                N.gemv_act(xa, mix.w_in, proj)
            else:
                N.gemv_post_norm(y, owed, c.eps, x, x2, mix.w_in, proj, next_norm=L["norm1"])
                x, x2 = x2, x
            mix.decode(lat, n, B.rotary.get(s.rot_dims, s.rot_base), pos, slot, self.page_table, c.eps, st)
            N.gemv_act(lat.mixed[s.heads * s.vdim][:n], mix.w_o, y)
            owed = L["norm1b"]
            if ff is not None:
                ff.decode(B.experts, n, y, owed, L["norm2"], c.eps, x, x2, xa, self.fabric.ticket_ptr)
                x, x2 = x2, x
                owed = L["norm2b"]
        N.post_norm_add(y, owed, c.eps, x, xa, self.final_norm)


class PonenexRows(StreamRows):
    """Packed-step executor: see :class:`StreamRows`."""
