from pace_b200.llm.models import garupel, gekupel, lesosun, llama  # noqa: F401  (registers the architectures)
