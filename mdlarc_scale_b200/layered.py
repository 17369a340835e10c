"""Layered models on the engine: the network as data, its session (cache, recurrent state, slots) and the
packing of mixed batches of prompt portions and single tokens."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np
import torch

from . import _lib
from .engine import EngineBase, Session, _ptr, _stream_ptr

QBLOCK = 256    # query rows of one tile pair of the prefill attention


@dataclass(frozen=True)
class LayerSpec:
    """One layer: a token mixer and an optional feed-forward (``arcb_layer_desc``)."""
    mixer: str                  # "attention" | "mlstm"
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    kv_from: int = -1
    qkv_bias: bool = False
    qk_norm: bool = False
    sink: bool = False
    out_gate: bool = False
    scale: float = 1.0
    q_temp_coef: float = 0.0
    q_temp_every: int = 0
    gate_cap: float = 1.0
    mlp: str | None = None      # "relu2" | None
    d_ff: int = 0


@dataclass(frozen=True)
class ModelSpec:
    width: int
    vocab: int
    layers: list[LayerSpec]
    norm: str = "layer"         # "layer" | "rms"
    norm_eps: float = 1e-6
    residual_alpha: float = 1.0
    logit_scale: float = 1.0


class LayeredEngine(EngineBase):
    """Packed weights of a layered model.  ``tensors`` maps (kind, layer) to fp32-convertible tensors in
    [out, in] order; the kinds are those of ``_lib.LAYERED_KINDS``."""

    end_token = -1

    def __init__(self, spec: ModelSpec, tensors: dict[tuple[str, int], torch.Tensor], device="cuda:0",
                 act_format: str = "f16", gemm_path: str = "auto", attn_path: str = "auto", mlstm_path: str = "auto",
                 fused_proj: bool = True):
        super().__init__(device)
        self.spec = spec
        self.vocab_size = spec.vocab
        self.n_layers = len(spec.layers)
        self.act_format = {"f16": _lib.ACT_F16, "bf16": _lib.ACT_BF16, "f32": _lib.ACT_F32}[act_format]
        md = _lib.ModelDesc(
            width=spec.width, vocab=spec.vocab, n_layers=self.n_layers, norm=_lib.NORMS[spec.norm],
            act_format=self.act_format, gemm_path={"auto": _lib.GEMM_AUTO, "simt": _lib.GEMM_SIMT}[gemm_path],
            attn_path={"auto": _lib.ATTN_AUTO, "stream": _lib.ATTN_STREAM}[attn_path],
            mlstm_path={"auto": _lib.MLSTM_AUTO, "step": _lib.MLSTM_STEP}[mlstm_path], fused_proj=int(bool(fused_proj)),
            norm_eps=spec.norm_eps, residual_alpha=spec.residual_alpha, logit_scale=spec.logit_scale)
        ld = (_lib.LayerDesc * self.n_layers)(*[
            _lib.LayerDesc(
                mixer=_lib.MIXERS[s.mixer], heads=s.heads, kv_heads=s.kv_heads, dim=s.dim, vdim=s.vdim, kv_from=s.kv_from,
                qkv_bias=int(s.qkv_bias), qk_norm=int(s.qk_norm), sink=int(s.sink), out_gate=int(s.out_gate),
                scale=s.scale, q_temp_coef=s.q_temp_coef, q_temp_every=s.q_temp_every, gate_cap=s.gate_cap,
                mlp=_lib.MLPS[s.mlp], d_ff=s.d_ff) for s in spec.layers])
        with torch.cuda.device(self.device):
            _lib.check(self.lib.arcb_engine_create_layered(C.byref(md), ld, C.byref(self._handle)))
            for (kind, layer), t in tensors.items():
                self._load_id(_lib.LAYERED_KIND[kind], layer, t)
            torch.cuda.synchronize(self.device)


@dataclass
class Segment:
    """The next tokens of the sequence in ``slot``; ``want``: places among them whose logits are asked for."""
    slot: int
    tokens: list[int] | np.ndarray
    want: list[int] = field(default_factory=list)
    arm: bool = False           # pick the first generated token from the last row and start decoding


@dataclass
class PackedSegments:
    """One prefill call's integer arrays, laid out in one host buffer that reaches the device in one copy."""
    buf: torch.Tensor
    at: dict[str, tuple[int, int]]
    n_tokens: int
    n_segs: int
    n_want: int
    n_first: int
    n_qblocks: int

    def ptr(self, dev: torch.Tensor, name: str) -> int | None:
        lo, n = self.at[name]
        return dev.data_ptr() + 4 * lo if n else None


def pack_segments(segments: list[Segment], pos0: list[int]) -> PackedSegments:
    """Packs portions of several sequences back to back.  Row arrays: token, cache row, position (= cache
    slot) and visible keys; segment arrays; the rows asked for; and the query blocks of the prefill
    attention, most expensive first (their CTAs are dispatched in that order)."""
    rows = np.array([len(s.tokens) for s in segments], np.int64)
    row0 = np.concatenate([[0], np.cumsum(rows)[:-1]]).astype(np.int64)
    slot = np.array([s.slot for s in segments], np.int64)
    p0 = np.array(pos0, np.int64)
    seg_of = np.repeat(np.arange(len(segments)), rows)
    pos = np.arange(int(rows.sum())) - row0[seg_of] + p0[seg_of]
    want = [int(row0[i]) + int(w) for i, s in enumerate(segments) for w in s.want]
    for i, s in enumerate(segments):
        if any(w < 0 or w >= rows[i] for w in s.want):
            raise ValueError("a wanted place lies outside its portion")
    arm = [i for i, s in enumerate(segments) if s.arm]
    blocks = [(int(row0[i]) + r, int(min(QBLOCK, rows[i] - r))) for i in range(len(segments)) for r in range(0, int(rows[i]), QBLOCK)]
    blocks.sort(key=lambda b: -int(pos[b[0] + b[1] - 1]))
    arrays = {
        "token": np.concatenate([np.asarray(s.tokens, np.int64) for s in segments]),
        "seq": slot[seg_of], "pos": pos, "count": pos + 1,
        "seg_row0": row0, "seg_rows": rows, "seg_seq": slot, "seg_pos0": p0,
        "want": want, "first_row": [int(row0[i] + rows[i] - 1) for i in arm], "first_seq": slot[arm] if arm else [],
        "first_len": [int(p0[i] + rows[i]) for i in arm],
        "qb_row0": [b[0] for b in blocks], "qb_rows": [b[1] for b in blocks],
    }
    at, parts, off = {}, [], 0
    for name, v in arrays.items():
        v = np.asarray(v, np.int32)
        at[name] = (off, len(v))
        pad = -len(v) % 4                     # every array starts on a 16-byte boundary
        parts.append(v)
        if pad:
            parts.append(np.zeros(pad, np.int32))
        off += len(v) + pad
    return PackedSegments(torch.from_numpy(np.concatenate(parts)), at, int(rows.sum()), len(segments), len(want),
                          len(arm), len(blocks))


class LayeredSession(Session):
    """Session of a layered model: slots of a cache that holds keys, values and recurrent states, all
    continued from call to call.  ``lens[slot]`` is the number of positions the slot holds."""

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self.lens = [0] * self.n_seqs
        self._free = list(range(self.n_seqs - 1, -1, -1))
        self._held: list = []
        if self.step_logits is not None and self.palette_mask is not None:
            raise ValueError("grid constraints do not apply to layered models")

    # -- slots ----------------------------------------------------------------
    def acquire(self) -> int:
        if not self._free:
            raise RuntimeError("no free slot in the session")
        slot = self._free.pop()
        self.lens[slot] = 0
        return slot

    def release(self, slot: int) -> None:
        if slot in self._free:
            raise ValueError(f"slot {slot} is already free")
        self.lens[slot] = 0
        self._free.append(slot)

    @property
    def free_slots(self) -> int:
        return len(self._free)

    # -- compute --------------------------------------------------------------
    def _check(self, slot: int, n: int) -> None:
        if slot < 0 or slot >= self.n_seqs:
            raise ValueError(f"slot {slot} outside the session")
        if n <= 0:
            raise ValueError("a portion must have at least one token")
        if self.lens[slot] + n > self.t_max:
            raise ValueError(f"slot {slot} would hold {self.lens[slot] + n} positions, the session has {self.t_max}")

    def prefill_segments(self, segments: list[Segment], logits_all: bool = False, residuals: bool = False):
        """One forward over portions of one or more sequences.  Returns (logits of the wanted rows in
        segment order or of all rows, first-token logits of the armed segments, residual stream after every
        layer), each None when not asked for."""
        slots = [s.slot for s in segments]
        if len(set(slots)) != len(slots):
            raise ValueError("a sequence may appear once in a call")
        for s in segments:
            self._check(s.slot, len(s.tokens))
        p = pack_segments(segments, [self.lens[s.slot] for s in segments])
        if p.n_tokens > self.max_prefill_tokens:
            raise ValueError("the call has more tokens than the session's prefill capacity")
        dev, V = self.eng.device, self.eng.vocab_size
        buf = p.buf.to(dev, non_blocking=True)
        f32 = dict(dtype=torch.float32, device=dev)
        everything = torch.empty((p.n_tokens, V), **f32) if logits_all else None
        wanted = torch.empty((p.n_want, V), **f32) if p.n_want else None
        first = torch.empty((p.n_first, V), **f32) if p.n_first else None
        res = torch.empty((self.eng.n_layers, p.n_tokens, self.eng.spec.width), **f32) if residuals else None
        a = _lib.PrefillArgs(
            n_tokens=p.n_tokens, d_token_ids=p.ptr(buf, "token"), d_seq=p.ptr(buf, "seq"), d_kv_slot=p.ptr(buf, "pos"),
            d_kv_count=p.ptr(buf, "count"), n_qblocks=p.n_qblocks, d_qblock_row0=p.ptr(buf, "qb_row0"),
            d_qblock_rows=p.ptr(buf, "qb_rows"), d_logits_all=_ptr(everything), n_first=p.n_first,
            d_first_row=p.ptr(buf, "first_row"), d_first_seq=p.ptr(buf, "first_seq"), d_prompt_len=p.ptr(buf, "first_len"),
            d_first_logits=_ptr(first), n_segs=p.n_segs, d_seg_row0=p.ptr(buf, "seg_row0"), d_seg_rows=p.ptr(buf, "seg_rows"),
            d_seg_seq=p.ptr(buf, "seg_seq"), d_seg_pos0=p.ptr(buf, "seg_pos0"), n_logit_rows=p.n_want,
            d_logit_row=p.ptr(buf, "want"), d_logits=_ptr(wanted), d_residuals=_ptr(res))
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_prefill(self._handle, C.byref(a), _stream_ptr(dev)))
        for s in segments:
            self.lens[s.slot] += len(s.tokens)
        return (everything if logits_all else wanted), first, res

    def feed(self, slots: list[int], tokens: list[int]) -> torch.Tensor:
        """One decode step (the captured graph) with the given tokens for the given slots; all other slots
        hold still.  Returns the step's logits [len(slots), vocab]."""
        if len(set(slots)) != len(slots):
            raise ValueError("a sequence may appear once in a step")
        for s in slots:
            self._check(s, 1)
        dev = self.eng.device
        buf = torch.tensor([*slots, *tokens], dtype=torch.int32).to(dev, non_blocking=True)
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_session_feed(self._handle, len(slots), buf.data_ptr(),
                                                      buf.data_ptr() + 4 * len(slots), _stream_ptr(dev)))
        self.decode(1)
        for s in slots:
            self.lens[s] += 1
        return self.last_logits()[buf[:len(slots)].long()]

    def last_logits(self) -> torch.Tensor:
        """View of the last decode step's logits, [n_seqs, vocab]; the next call overwrites it."""
        ptr, pitch = C.c_void_p(), C.c_int32()
        _lib.check(self.eng.lib.arcb_session_step_logits(self._handle, C.byref(ptr), C.byref(pitch)))
        off = ptr.value - self.workspace.data_ptr()
        rows = self.workspace[off:off + self.n_seqs * pitch.value * 4].view(torch.float32)
        return rows.view(self.n_seqs, pitch.value)[:, :self.eng.vocab_size]

    def step(self, segments: list[Segment]) -> list[torch.Tensor | None]:
        """Advances every named sequence by its portion: single tokens of started sequences through the decode
        step, anything else through prefill.  Per segment the logits of its wanted places (or None)."""
        if all(len(s.tokens) == 1 and self.lens[s.slot] > 0 for s in segments):
            rows = self.feed([s.slot for s in segments], [int(s.tokens[0]) for s in segments])
            return [rows[i:i + 1].clone() if s.want else None for i, s in enumerate(segments)]
        out: list[list[torch.Tensor]] = [[] for _ in segments]
        done = [0] * len(segments)
        while True:
            call, owner, room = [], [], self.max_prefill_tokens
            for i, s in enumerate(segments):
                n = min(len(s.tokens) - done[i], room)
                if n > 0:
                    want = [w - done[i] for w in s.want if done[i] <= w < done[i] + n]
                    call.append(Segment(s.slot, s.tokens[done[i]:done[i] + n], want, s.arm and done[i] + n == len(s.tokens)))
                    owner.append(i)
                    done[i] += n
                    room -= n
            if not call:
                break
            logits, _, _ = self.prefill_segments(call)
            at = 0
            for i, c in zip(owner, call):
                if c.want:
                    out[i].append(logits[at:at + len(c.want)])
                    at += len(c.want)
        return [torch.cat(o) if o else None for o in out]

    def finished(self) -> np.ndarray:
        """Flags of the slots that have emitted the end token or used up ``max_new`` (synchronises)."""
        flags = np.zeros(self.n_seqs, np.int32)
        dev = self.eng.device
        with torch.cuda.device(dev):
            _lib.check(self.eng.lib.arcb_session_finished(self._handle, flags.ctypes.data, _stream_ptr(dev)))
        return flags


LayeredEngine.session_class = LayeredSession
