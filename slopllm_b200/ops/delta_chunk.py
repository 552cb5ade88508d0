"""Chunked form of the channel-wise gated delta rule (see `ops/delta.py`)."""


def usable(s, plan, out) -> bool:
    return False


def run(*a):
    raise NotImplementedError
