"""Python face of the served-model interface (``tm_model_*``): open a checkpoint folder, prefill, decode, and the scheduler
over it (``llama.Batch`` takes these models too).  Everything that computes is in ``libtm_b200.so``.
"""
from __future__ import annotations

import ctypes as C
import json
from typing import Optional, Sequence

import torch

from . import lib as _l

DTYPES = {"bfloat16": _l.TM_DTYPE_BF16, "float32": _l.TM_DTYPE_F32}


def architectures():
    buf = C.create_string_buffer(1024)
    _l.check(_l.lib.tm_model_architectures(buf, len(buf)), "tm_model_architectures")
    return buf.value.decode().split(",")


def _ints(xs):
    return (C.c_int * max(1, len(xs)))(*[int(x) for x in xs])


class Model:
    """A tm_model: ``Model.open(folder)`` for a checkpoint, ``Model.random(config)`` for random weights."""

    def __init__(self, ptr: C.c_void_p, handle: "_l.Handle", device: int):
        self.ptr, self.handle, self.device = ptr, handle, device
        info = _l.TmModelInfo()
        _l.check(_l.lib.tm_model_describe(ptr, C.byref(info)), "tm_model_describe")
        self.vocab_size, self.max_batch_size, self.session_len = info.vocab_size, info.max_batch_size, info.session_len
        self.can_rewind, self.slab_bytes = bool(info.can_rewind), info.slab_bytes

    @classmethod
    def open(cls, folder: str, dtype: str = "bfloat16", max_batch_size: int = 32, session_len: int = 4096, max_prefill_tokens: int = 0,
             device: int = 0) -> "Model":
        return cls._make(lambda p, h, o: _l.lib.tm_model_open(p, h, folder.encode(), o), f"tm_model_open({folder})", dtype, max_batch_size,
                         session_len, max_prefill_tokens, device)

    @classmethod
    def random(cls, config: dict, dtype: str = "bfloat16", max_batch_size: int = 32, session_len: int = 4096, max_prefill_tokens: int = 0,
               device: int = 0, seed: int = 0) -> "Model":
        text = json.dumps(config).encode()
        return cls._make(lambda p, h, o: _l.lib.tm_decoder_create_random(p, h, text, o, seed), "tm_decoder_create_random", dtype,
                         max_batch_size, session_len, max_prefill_tokens, device)

    @classmethod
    def _make(cls, call, what, dtype, max_batch_size, session_len, max_prefill_tokens, device):
        handle = _l.default_handle(device)
        opt = _l.TmModelOptions(DTYPES[dtype], max_batch_size, session_len, max_prefill_tokens)
        ptr = C.c_void_p()
        rc = call(C.byref(ptr), handle.ptr, C.byref(opt))
        if rc != _l.TM_OK:
            raise _l.TmError(rc, f"{what}: {_l.lib.tm_model_last_error().decode()}")
        return cls(ptr, handle, device)

    def new_cache(self, max_entry_count: int, chunk_size: int = 1) -> C.c_void_p:
        cache = C.c_void_p()
        _l.check(_l.lib.tm_model_new_cache(self.ptr, max_entry_count, chunk_size, C.byref(cache)), "tm_model_new_cache")
        return cache

    def prefill(self, tokens: Sequence[Sequence[int]], histories: Sequence[int], slabs: Sequence[int],
                want: Optional[Sequence[Sequence[int]]] = None, residual: bool = False, layers: int = 0, width: int = 0):
        """New tokens per sequence on top of ``histories``; ``slabs`` are device addresses.  -> (logits of the wanted
        places, in order, or None; residual stream [layers, tokens, width] or None)"""
        cu, packed, wanted = [0], [], []
        for b, t in enumerate(tokens):
            wanted += [cu[-1] + w for w in (want[b] if want else [])]
            packed += list(t)
            cu.append(len(packed))
        dev = torch.device("cuda", self.device)
        logits = torch.empty(len(wanted), self.vocab_size, device=dev) if wanted else None
        res = torch.empty(layers, len(packed), width, device=dev) if residual else None
        st = _l.TmModelPrefillState()
        ptrs = (C.c_void_p * len(slabs))(*slabs)
        keep = (_ints(packed), _ints(cu), _ints(histories), _ints(wanted))
        st.batch_size, st.input_ids, st.cu_seqlens, st.history_lengths = len(tokens), keep[0], keep[1], keep[2]
        st.k_cache, st.v_cache = ptrs, ptrs
        st.want_count, st.want = len(wanted), keep[3]
        st.logits_out = 0 if logits is None else logits.data_ptr()
        st.residual_out = 0 if res is None else res.data_ptr()
        _l.check(_l.lib.tm_model_prefill(self.ptr, C.byref(st), torch.cuda.current_stream().cuda_stream), "tm_model_prefill")
        return logits, res

    def new_state(self, slabs: Sequence[int], lengths: Sequence[int], max_steps: int = 1, forced_ids=None, start_step=None) -> "DecodeState":
        return DecodeState(self, slabs, lengths, max_steps, forced_ids, start_step)

    def decode(self, state: "DecodeState", n_steps: int = 1, use_graph: bool = False, stream=None) -> None:
        s = torch.cuda.current_stream().cuda_stream if stream is None else stream
        _l.check(_l.lib.tm_model_decode(self.ptr, C.byref(state.c), n_steps, int(use_graph), s), "tm_model_decode")

    def check_status(self) -> None:
        w = C.c_uint(0)
        rc = _l.lib.tm_model_check_status(self.ptr, torch.cuda.current_stream().cuda_stream, C.byref(w))
        if rc != _l.TM_OK:
            raise _l.TmError(rc, f"tm_model_check_status: device status word 0x{w.value:x}")

    def last_launches(self) -> int:
        return int(_l.lib.tm_model_last_launches(self.ptr))

    def close(self):
        if self.ptr:
            _l.lib.tm_model_close(self.ptr)
            self.ptr = C.c_void_p()


class DecodeState:
    """Device buffers of a ``tm_llama_decode_state`` over slabs of a served model."""

    def __init__(self, model: Model, slabs, lengths, max_steps, forced_ids, start_step):
        dev, b = torch.device("cuda", model.device), len(slabs)
        self.ptrs = torch.tensor(list(slabs), dtype=torch.int64, device=dev)
        self.lengths = torch.tensor(list(lengths), dtype=torch.int32, device=dev)
        self.step = torch.zeros(1, dtype=torch.int32, device=dev)
        self.output_ids = torch.full((max_steps, b), -1, dtype=torch.int32, device=dev)
        self.forced_ids = None if forced_ids is None else torch.as_tensor(forced_ids, dtype=torch.int32).to(dev).contiguous()
        self.start_step = None if start_step is None else torch.as_tensor(start_step, dtype=torch.int32).to(dev)
        self.logits = torch.zeros(b, model.vocab_size, device=dev)
        c = _l.TmLlamaDecodeState()
        c.batch_size, c.max_steps = b, max_steps
        c.k_cache_ptrs = c.v_cache_ptrs = self.ptrs.data_ptr()
        c.sequence_lengths, c.step, c.output_ids = self.lengths.data_ptr(), self.step.data_ptr(), self.output_ids.data_ptr()
        c.forced_ids = 0 if self.forced_ids is None else self.forced_ids.data_ptr()
        c.start_step = 0 if self.start_step is None else self.start_step.data_ptr()
        c.logits_out = self.logits.data_ptr()
        self.c = c
