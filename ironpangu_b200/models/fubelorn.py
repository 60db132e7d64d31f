"""Fubelorn: a decoder whose residual is several streams side by side (hyper-connections with fixed weights, f32) and whose sublayers read the norm of
their weighted sum with a short causal convolution over it: h = rms(sum in_s x_s) g, operand h + conv(h), x_t <- sum mix_st x_s + mult out_t y.

  parallel      left_scale * attention + right_scale * recurrence of the same operand: grouped heads over a window and the first ``mask.keep_first``
                positions, every head of q and k by its rms, no rotation; beside it the gated delta rule
  mamba2        state-space duality: z | x | B | C | dt projected together, x B C convolved, y + D x gated by silu(z) and normed in groups
  parallel_2    grouped heads over a window and the means of blocks of ``mask.pool`` positions ahead of it, rotated halves with stretched
                wavelengths, a gate per head; beside it a matrix memory with exponential gates
  dense         W_down gelu(W_up h), exact GELU

Norms have one number for all columns. ``FubelornDecoder`` and ``FubelornRows`` are the decode and packed-step executors (``stream_decoder.py``).
In bf16 the linears take bf16 operands with f32 accumulation; streams, norms, rotations, scores, gates and recurrences are f32. With
``dtype=torch.float32`` every product is a true f32 FMA.

A checkpoint directory is ``config.json`` (``"architecture": "Fubelorn"``) + safetensors; see :func:`weight_shapes` for the names."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from ..ops import hyper_streams as HS
from ..ops import stream_norm as N
from ..ops.gated_recurrence import CHUNK, TILE, GatedRecurrence, RecurrenceBuffers, RecurrenceShape
from ..ops.linear_attn import DevicePlan, RotaryScaling, RotaryTables
from ..ops.window_attn import GroupedAttention, GroupedBuffers, GroupedShape
from ..parallel.fabric import Fabric
from . import checkpoint
from .checkpoint import pad8
from .stream_decoder import ATTN_ROWS, BF16, F32, StreamDecoder, StreamRows

KERNEL_UNITS = ("misc", "post_norm", "hyper_streams", "gated_recurrence", "gated_delta", "gated_tiles", "linear_f32", "window_attn", "decode_gqa", "fa_prefill", "decode_post_norm",
                "decode_hyper", "decode_moe", "sampling", "tc_gemm", "tc_gemm_2sm")
MIXERS = ("parallel", "mamba2", "parallel_2")


# ---------------------------------------------------------------------------------------------------------------------------
# configuration
# ---------------------------------------------------------------------------------------------------------------------------
@dataclass
class LayerConfig:
    """``right``: the recurrence, alone or beside the attention ``left``."""

    kind: str
    right: RecurrenceShape
    left: Optional[GroupedShape] = None
    right_scale: float = 1.0             # the attention's is its shape's factor
    ff: int = 0                          # 0: no feed-forward

    @property
    def in_cols(self) -> int:
        """Columns of the packed projection [attention | recurrence], filled up to whole stores of the GEMMs."""
        return ((self.left.in_cols if self.left else 0) + self.right.in_cols + 31) // 32 * 32

    @property
    def right_at(self) -> int:
        return self.left.in_cols if self.left else 0

    @property
    def mixed(self) -> tuple:
        """Columns of the operand of the output projection: the attention's (padded) and the recurrence's."""
        return pad8(self.left.heads * self.left.vdim) if self.left else 0, pad8(self.right.inner)


@dataclass
class FubelornConfig:
    vocab: int
    width: int
    eps: float
    streams: int                         # 0: a plain residual
    mult: float
    taps: int                            # of the convolution ahead of every sublayer (0: none)
    layers: List[LayerConfig] = field(default_factory=list)
    page_tokens: int = 16

    @staticmethod
    def from_dict(j: dict) -> "FubelornConfig":
        if j.get("architecture") != "Fubelorn":
            raise ValueError(f"not a Fubelorn configuration (architecture {j.get('architecture')!r})")
        layers = []
        for i, e in enumerate(j["layers"]):
            m, f, kind = e["mixer"], e.get("mlp"), e["type"]
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            if f is not None and f.get("kind") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f.get('kind')!r}")
            ff = int(f["ff"]) if f is not None else 0
            if kind == "mamba2":
                layers.append(LayerConfig(kind, RecurrenceShape("ssd", int(m["heads"]), int(m["groups"]), int(m["state"]), int(m["vdim"]), int(m["conv"]), int(m["norm_groups"])),
                                          ff=ff))
                continue
            l, r = m["left"], m["right"]
            mask = l.get("mask") or {}
            sizes = dict(heads=int(l["heads"]), kv_heads=int(l["kv_heads"]), dim=int(l["dim"]), vdim=int(l["vdim"]), scale=float(l["scale"]), window=int(mask.get("size", 0)),
                         factor=float(m["left_scale"]))
            if kind == "parallel":
                left = GroupedShape(**sizes, keep=int(mask.get("keep_first", 0)), head_norm=True, gated=False)
                right = RecurrenceShape("delta", int(r["heads"]), int(r["kv_heads"]), int(r["dim"]), int(r["vdim"]), int(r["conv"]))
            else:
                rot = l.get("rot") or {}
                sc = rot.get("scaling")
                scaling = RotaryScaling(*(float(sc[n]) for n in ("factor", "low", "high", "original"))) if sc else None
                left = GroupedShape(**sizes, pool=int(mask.get("pool", 0)), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), rot_scaling=scaling,
                                    rot_halves=True)
                right = RecurrenceShape("memory", int(r["heads"]), int(r["heads"]), int(r["dim"]), int(r["vdim"]), gate_cap=float(r["gate_cap"]))
            layers.append(LayerConfig(kind, right, left, float(m["right_scale"]), ff))
        return FubelornConfig(int(j["vocab"]), int(j["width"]), float(j["norm"]["eps"]), int(j.get("streams") or 0), float(j.get("residual_mult", 1.0)),
                              int((j.get("canon") or {}).get("taps", 0)), layers).validate()

    def to_dict(self) -> dict:
        out = []
        for c in self.layers:
            l, r = c.left, c.right
            if c.kind == "mamba2":
                m = {"heads": r.heads, "groups": r.kv_heads, "state": r.dim, "vdim": r.vdim, "conv": r.taps, "norm_groups": r.norm_groups}
            else:
                left = {"heads": l.heads, "kv_heads": l.kv_heads, "dim": l.dim, "vdim": l.vdim, "scale": l.scale, "mask": {"size": l.window}}
                right = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim}
                if c.kind == "parallel":
                    left["mask"]["keep_first"] = l.keep
                    right.update(kv_heads=r.kv_heads, conv=r.taps)
                else:
                    left["mask"]["pool"] = l.pool
                    s = l.rot_scaling
                    left["rot"] = {"dims": l.rot_dims, "base": l.rot_base, **({"scaling": {"factor": s.factor, "low": s.low, "high": s.high, "original": s.original}} if s else {})}
                    right["gate_cap"] = r.gate_cap
                m = {"left": left, "right": right, "left_scale": l.factor, "right_scale": c.right_scale}
            out.append({"type": c.kind, "mixer": m, "mlp": {"kind": "dense", "ff": c.ff} if c.ff else None})
        return {"architecture": "Fubelorn", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "streams": self.streams, "residual_mult": self.mult,
                "canon": {"taps": self.taps}, "layers": out}

    def validate(self) -> "FubelornConfig":
        if not self.layers:
            raise ValueError("no layers")
        if not 0 <= self.streams <= HS.MOST_STREAMS or not 0 <= self.taps <= HS.MOST_TAPS or max(self.taps, 1) * self.width > 50000:
            raise ValueError(f"{self.streams} streams, a convolution of {self.taps} taps over {self.width} columns are not supported")
        for i, l in enumerate(self.layers):
            try:
                l.right.check()
                if l.left:
                    l.left.check()
            except ValueError as e:
                raise ValueError(f"layer {i}: {e}") from None
        return self

    @property
    def window(self) -> int:
        """How far back any layer reads the pages when every layer has a limit, else 0: kept first positions and blocks ahead of a window keep them all."""
        w = [0 if l.left.keep or l.left.pool else l.left.window for l in self.layers if l.left]
        return max(w) if w and all(w) else 0

    def param_count(self) -> int:
        return checkpoint.param_count(weight_shapes(self))

    @staticmethod
    def tiny() -> "FubelornConfig":
        """Every mixer in unequal sizes, a layer without a feed-forward, three streams; odd sizes."""
        a = GroupedShape(6, 2, 40, 24, 0.2, 20, keep=3, head_norm=True, gated=False, factor=0.7)
        b = GroupedShape(4, 4, 24, 56, 0.3, 24, pool=5, rot_dims=16, rot_base=1e5, rot_scaling=RotaryScaling(4.0, 1.0, 4.0, 64.0), rot_halves=True, factor=1.2)
        delta, memory = RecurrenceShape("delta", 6, 3, 16, 40, 4), RecurrenceShape("memory", 3, 3, 24, 40, gate_cap=12.0)
        ssd = RecurrenceShape("ssd", 4, 2, 24, 48, 4, 2)
        return FubelornConfig(384, 136, 1e-5, 3, 0.8, 3, [LayerConfig("parallel", delta, a, 1.1, 200), LayerConfig("mamba2", ssd, ff=120), LayerConfig("parallel_2", memory, b, 0.9),
                                                          LayerConfig("mamba2", ssd, ff=200)]).validate()

    @staticmethod
    def text(layers: int = 16, width: int = 2048, heads: int = 16, kv_heads: int = 4, dim: int = 128, ff: int = 6144, vocab: int = 128000, window: int = 1024, keep: int = 16,
             pool: int = 16, rec_heads: int = 8, rec_dim: int = 128, state: int = 128, streams: int = 2) -> "FubelornConfig":
        """(parallel, mamba2, parallel_2, mamba2) repeated."""
        a = GroupedShape(heads, kv_heads, dim, dim, dim ** 0.5 / 4, window, keep=keep, head_norm=True, gated=False, factor=0.7)
        b = GroupedShape(heads, kv_heads, dim, dim, dim ** -0.5, window, pool=pool, rot_dims=dim, rot_base=5e5, rot_scaling=RotaryScaling(8.0, 1.0, 4.0, 8192.0), rot_halves=True,
                         factor=0.7)
        delta, memory = RecurrenceShape("delta", rec_heads, rec_heads, rec_dim, rec_dim, 4), RecurrenceShape("memory", rec_heads, rec_heads, rec_dim, rec_dim, gate_cap=15.0)
        ssd = RecurrenceShape("ssd", 2 * width // 128, 1, state, 128, 4, 1)
        kinds = (LayerConfig("parallel", delta, a, 0.7, ff), LayerConfig("mamba2", ssd, ff=ff), LayerConfig("parallel_2", memory, b, 0.7, ff), LayerConfig("mamba2", ssd, ff=ff))
        return FubelornConfig(vocab, width, 1e-6, streams, 1.0, 4, [kinds[i % 4] for i in range(layers)]).validate()


PRESETS = {"fubelorn-tiny": FubelornConfig.tiny, "fubelorn-text": FubelornConfig.text}


# ---------------------------------------------------------------------------------------------------------------------------
# weights
# ---------------------------------------------------------------------------------------------------------------------------
def weight_shapes(c: FubelornConfig) -> Dict[str, tuple]:
    """Checkpoint tensor names -> shapes (bf16 in the file)."""
    W = c.width
    s = {"embed": (c.vocab, W), "embed.norm": (), "final.norm": (), "head": (c.vocab, W)}
    for i, y in enumerate(c.layers):
        p, l, r = f"l{i}.", y.left, y.right
        qk, v, h = r.kv_heads * r.dim, r.inner, r.heads
        m = p + "mix." + ("right." if l else "")
        if l:
            n = p + "mix.left."
            s.update({n + "q": (l.heads * l.dim, W), n + "k": (l.kv_heads * l.dim, W), n + "v": (l.kv_heads * l.vdim, W), n + "o": (W, l.heads * l.vdim)})
            if l.gated:
                s[n + "g"] = (l.heads, W)
        if r.kind == "ssd":
            s.update({m + "in": (r.in_cols, W), m + "conv": (r.channels, r.taps), m + "conv.b": (r.channels,), m + "D": (h,), m + "norm": (v,)})
        else:
            s.update({m + "q": (qk, W), m + "k": (qk, W), m + "v": (v, W), m + "g": (v, W), m + "norm": (r.vdim if r.kind == "delta" else v,)})
        if r.kind == "delta":
            s.update({m + "q.conv": (qk, r.taps), m + "k.conv": (qk, r.taps), m + "v.conv": (v, r.taps), m + "a": (h, W), m + "b": (h, W)})
        if r.kind == "memory":
            s.update({m + "i": (h, W), m + "i.b": (h,), m + "f": (h, W), m + "f.b": (h,)})
        else:
            s.update({m + "A_log": (h,), m + "dt_bias": (h,)})
        s[m + "o"] = (W, v)
        if y.ff:
            s.update({p + "mlp.up": (y.ff, W), p + "mlp.down": (W, y.ff)})
        for q in (1, 2) if y.ff else (1,):
            s[f"{p}norm{q}"] = ()
            if c.streams:
                s.update({f"{p}hc{q}.in": (c.streams,), f"{p}hc{q}.out": (c.streams,), f"{p}hc{q}.mix": (c.streams, c.streams)})
            if c.taps:
                s[f"{p}canon{q}"] = (W, c.taps)
    return s


def random_weights(c: FubelornConfig, device, seed: int = 0, std: float = 0.02) -> Dict[str, torch.Tensor]:
    """Random-init checkpoint tensors: N(0, std) matrices and biases, gains 1 + N(0, std), taps N(0, 1 / taps), streams mixed by a perturbed identity, decays of
    many lengths."""
    g = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        t = torch.empty(shape, dtype=F32, device=device).normal_(0.0, std, generator=g)
        if "norm" in name or name.endswith((".D", "hc1.out", "hc2.out")):
            t += 1.0
        elif "canon" in name or name.endswith("conv"):
            t *= (1.0 / shape[1]) ** 0.5 / std
        elif name.endswith(".mix"):
            t += torch.eye(shape[0], device=device)
        elif name.endswith(("hc1.in", "hc2.in")):
            t += 1.0 / shape[0]
        elif name.endswith("A_log"):
            t = torch.linspace(0.0, 2.0, shape[0], device=device)
        elif name.endswith("dt_bias"):
            t += torch.linspace(-5.0, -2.0, shape[0], device=device)
        elif name.endswith("f.b"):
            t += torch.linspace(2.0, 5.0, shape[0], device=device)
        out[name] = t.to(BF16)
    return out


def save_checkpoint(path, c: FubelornConfig, weights: Dict[str, torch.Tensor]) -> None:
    checkpoint.save(path, c, weights)


def load_checkpoint(path) -> tuple:
    """``(config, weights on the host)`` of a checkpoint directory; every expected tensor must be there with its shape."""
    return checkpoint.load(path, FubelornConfig.from_dict, weight_shapes)


# ---------------------------------------------------------------------------------------------------------------------------
# executors
# ---------------------------------------------------------------------------------------------------------------------------
class _Rows:
    """Step buffers for up to ``rows`` rows (leading dimensions padded to 8 elements, padding zero)."""

    def __init__(self, dec: "FubelornDecoder", rows: int, chunked: bool):
        c, dev, A = dec.cfg, dec.fabric.device, dec.dtype
        z = lambda n, dt=A: torch.zeros(rows, pad8(n), dtype=dt, device=dev)
        self.rows = rows
        self.x, self.xa, self.y = z(c.width, F32), z(c.width), z(c.width, F32)           # sum of the streams (first the embedding), operand, sublayer result
        self.streams = [torch.zeros(rows, max(c.streams, 1), pad8(c.width), dtype=F32, device=dev) for _ in range(2)]
        left = [l.left for l in c.layers if l.left]
        self.attn = GroupedBuffers(left, rows, A, dev, chunked=chunked, max_context=dec.max_context, group=ATTN_ROWS, in_cols=max(l.in_cols for l in c.layers))
        self.rec = RecurrenceBuffers([l.right for l in c.layers], rows, A, dev, chunk=dec.chunk if chunked else 0, slots=dec.num_slots)
        self.mixed = {l.mixed: z(sum(l.mixed)) for l in c.layers}                        # one per pair of widths: the padding columns must stay zero
        self.act = {l.ff: z(l.ff) for l in c.layers if l.ff}
        self.parts = torch.zeros(8, min(rows, 128), pad8(c.width), dtype=F32, device=dev) if A == BF16 else None
        self.rotary = RotaryTables([s.rotation for s in left], rows, dev)


class FubelornDecoder(StreamDecoder):
    """Decode executor: see :class:`StreamDecoder`."""

    name = "fubelorn"

    def make_rows(self, rows: int, chunked: bool) -> _Rows:
        return _Rows(self, rows, chunked)

    def _load(self, W: Dict[str, torch.Tensor]) -> None:
        c, dev = self.cfg, self.fabric.device
        self.embed, self.head = self._mat(W, "embed"), self._mat(W, "head")
        one = lambda n: W[n].to(dev).float().reshape(1)
        self.embed_gain, self.final_gain = one("embed.norm"), one("final.norm")
        self.final_norm = self.final_gain.repeat(c.width)
        self.layers: List[dict] = []
        for i, l in enumerate(c.layers):
            p = f"l{i}."
            n = p + "mix." + ("right." if l.left else "")
            left = GroupedAttention(l.left, W, p + "mix.left.", dev, self.dtype) if l.left else None
            right = GatedRecurrence(l.right, W, n, dev, self.dtype, at=l.right_at, factor=l.right_scale)
            w_in = torch.zeros(l.in_cols, pad8(c.width), dtype=self.dtype, device=dev)
            if left:
                w_in[:l.right_at] = left.w_in
                left.w_in = None
            w_in[l.right_at:l.right_at + l.right.in_cols, :c.width] = right.w_in
            right.w_in = None
            a, b = l.mixed
            w_out = torch.zeros(c.width, a + b, dtype=self.dtype, device=dev)
            if left:
                w_out[:, :l.left.heads * l.left.vdim] = W[p + "mix.left.o"].to(dev)
            w_out[:, a:a + l.right.inner] = W[n + "o"].to(dev)
            sub = [HS.Sublayer(W, p, q, c.streams, c.mult, c.taps, c.width, dev) for q in ((1, 2) if l.ff else (1,))]
            self.layers.append({"c": l, "left": left, "right": right, "in": w_in, "out": w_out, "sub": sub,
                                "up": self._mat(W, p + "mlp.up") if l.ff else None, "down": self._mat(W, p + "mlp.down") if l.ff else None})
        # prompts: recurrences on the tensor cores in bf16 when every head fits a tile, f32 products otherwise
        self.chunk = TILE if self.dtype == BF16 and all(l.right.tiles for l in c.layers) else CHUNK
        # the fused decode chain needs operand widths that are whole 16-byte chunks
        self.side = torch.cuda.Stream()
        self.fused = self.dtype == BF16 and c.streams <= HS.FUSED_STREAMS and c.width % 8 == 0 and c.width <= 8192 and all(l.ff % 8 == 0 for l in c.layers) and \
            all(L["right"].fusable for L in self.layers)

    def _state_bytes(self) -> tuple:
        c, es = self.cfg, torch.empty((), dtype=self.dtype).element_size()
        page = sum(l.left.page(c.page_tokens) for l in c.layers if l.left) * es
        slot = sum(4 * l.right.slot_floats + 2 * max(l.right.taps - 1, 0) * l.right.channels * es + 2 * max(c.taps - 1, 0) * c.width * 4 * (2 if l.ff else 1) for l in c.layers)
        return (page + c.page_tokens - 1) // c.page_tokens, slot

    def _make_states(self) -> None:
        c, dev = self.cfg, self.fabric.device
        self.epoch = torch.zeros(self.num_slots, dtype=torch.int32, device=dev)
        for L in self.layers:
            L["state"] = L["right"].make_state(self.num_slots, dev, self.dtype)
            L["pages"] = L["left"].make_pages(self.num_pages, c.page_tokens, dev, self.dtype) if L["left"] else None
            for s in L["sub"]:
                s.make_history(self.num_slots, c.width, dev)

    @classmethod
    def from_checkpoint(cls, path, fabric: Fabric, **kw) -> "FubelornDecoder":
        c, w = load_checkpoint(path)
        return cls(c, w, fabric, **kw)

    # -- layers ------------------------------------------------------------------------------------------------------------
    def _side_by_side(self, B: _Rows, L: dict, m: int, pos, slot, plan: Optional[DevicePlan], recurrence) -> torch.Tensor:
        """The mixer of one layer between its input projection (``B.attn.proj``) and the operand of its output projection, which it returns. A layer with an
        attention runs it beside ``recurrence(operand's second part)``, on a stream of its own between two events."""
        l = L["c"]
        out = B.mixed[l.mixed][:m]
        right = out[:, l.mixed[0]:]
        if l.left is None:
            recurrence(right)
            return out
        main = torch.cuda.current_stream()
        self.side.wait_stream(main)
        with torch.cuda.stream(self.side):
            recurrence(right)
        L["left"].attend(B.attn, m, L["pages"], B.rotary.get(*l.left.rotation), pos, slot, plan, self.page_table, self.cfg.eps, out, self.fabric.desc.status)
        main.wait_stream(self.side)
        return out

    def _mix(self, B: _Rows, L: dict, m: int, pos, slot, plan: Optional[DevicePlan]) -> torch.Tensor:
        run = lambda out: L["right"].mix(B.rec, L["state"], B.attn.proj[:m], pos, slot, plan, self.epoch, self.cfg.eps, out, self.fabric.desc.status)
        return self._side_by_side(B, L, m, pos, slot, plan, run)

    def _product(self, B: _Rows, x: torch.Tensor, w: torch.Tensor, m: int) -> torch.Tensor:
        """f32 rows ``x w^T``: in ``B.y``, or for few rows as parts of a sum ``[parts, m, width]``."""
        width, k = w.shape
        n = 1 if B.parts is None else N.split_count(m, width, k)
        if n == 1:
            N.linear(x, w, B.y[:m, :width], status_ptr=self.fabric.desc.status)
            return B.y[:m]
        parts = B.parts[:n, :m]
        N.split_linear(x, w, parts[:, :, :width], status_ptr=self.fabric.desc.status)
        return parts

    def _layers(self, B: _Rows, m: int, tok, pos, slot, plan: Optional[DevicePlan], final: bool, probe: Optional[list] = None) -> None:
        """All layers over ``m`` rows as separate row operators and matrix products; the sum of the streams ends in ``B.x``, and with ``final``
        the normalised rows for the output matrix in ``B.xa``."""
        c, st, W = self.cfg, self.fabric.desc.status, self.cfg.width
        x, xa = B.x[:m, :W], B.xa[:m]
        HS.step_epoch(slot, self.epoch)
        HS.embed_norm(tok, self.embed, self.embed_gain, c.eps, x, st)
        B.rotary.fill(pos)
        now, spare = x[:, None].expand(-1, max(c.streams, 1), -1), [t[:m, :, :W] for t in B.streams]
        before, y = None, None

        def front(after, **kw):
            """The streams behind the last sublayer and the operand of the next."""
            nonlocal now
            to = spare[0] if y is not None and after is not None else None
            HS.streams_rows(now, to, y, before, after, self.final_gain, c.eps, self.epoch, pos, slot, kw.pop("operand", xa), **kw)
            if to is not None:
                now = to
                spare.reverse()

        for L in self.layers:
            l = L["c"]
            front(L["sub"][0])
            N.linear(xa, L["in"], B.attn.proj[:m, :l.in_cols], status_ptr=st)
            y, before = self._product(B, self._mix(B, L, m, pos, slot, plan), L["out"], m), L["sub"][0]
            if l.ff:
                front(L["sub"][1])
                act = B.act[l.ff][:m]
                N.linear(xa, L["up"], act[:, :l.ff], "gelu_erf", status_ptr=st)
                y, before = self._product(B, act, L["down"], m), L["sub"][1]
            if probe is not None:                  # the sum of the streams as the layer leaves them
                t = torch.empty_like(x, memory_format=torch.contiguous_format)
                front(None, operand=None, total=t)
                probe.append(t)
        front(None, operand=xa if final else None, total=x)


    def _layers_fused(self, B: _Rows, n: int, tok, pos, slot) -> None:
        """One or two decode rows: streams, norm and convolution at the front of the linear that reads them, convolution, gates and step of a recurrence in one
        launch, its norm and gate at the front of the output projection. Ends like :meth:`_layers` with ``final``."""
        c, W = self.cfg, self.cfg.width
        x, y = B.x[:n, :W], B.y[:n]
        HS.step_epoch(slot, self.epoch)
        HS.embed_norm(tok, self.embed, self.embed_gain, c.eps, x, self.fabric.desc.status)
        B.rotary.fill(pos)
        now, spare = x[:, None].expand(-1, max(c.streams, 1), -1), [t[:n, :, :W] for t in B.streams]
        before = None
        for L in self.layers:
            l, proj = L["c"], B.attn.proj[:n]
            for sub, w, out, act in ((L["sub"][0], L["in"], proj, None),) + (((L["sub"][1], L["up"], B.act[l.ff][:n], "gelu_erf"),) if l.ff else ()):
                HS.gemv_streams(now, None if before is None else spare[0], None if before is None else y, before, sub, c.eps, self.epoch, pos, slot, w, out, act)
                if before is not None:
                    now = spare[0]
                    spare.reverse()
                before = sub
                if act is None:
                    mixed = self._side_by_side(B, L, n, pos, slot, None, lambda _: L["right"].decode(B.rec, L["state"], proj, pos, slot, self.epoch))
                    L["right"].gemv_mixed(B.rec, proj, c.eps, mixed, l.mixed[0], L["out"], y)
                else:
                    N.gemv_act(out, L["down"], y)
        HS.streams_rows(now, None, y, before, None, self.final_gain, c.eps, self.epoch, pos, slot, B.xa[:n], x)


class FubelornRows(StreamRows):
    """Packed-step executor: see :class:`StreamRows`."""
