// See json.h.
#include "json.h"
#include <cmath>
#include <cstdlib>
#include <cstring>
#include <stdexcept>

namespace mk {

class JsonReader {
public:
    JsonReader(const char* p, size_t n, const std::string& what) : p_(p), n_(n), what_(what) {}

    Json document() {
        Json v = value(what_, 0);
        space();
        if (at_ != n_) fail("text after the document");
        return v;
    }

private:
    [[noreturn]] void fail(const std::string& why) const {
        throw std::runtime_error(what_ + ": malformed JSON at byte " + std::to_string(at_) + ": " + why);
    }
    void space() {
        while (at_ < n_ && (p_[at_] == ' ' || p_[at_] == '\t' || p_[at_] == '\n' || p_[at_] == '\r')) ++at_;
    }
    char peek() {
        space();
        if (at_ >= n_) fail("unexpected end");
        return p_[at_];
    }
    void expect(char c) {
        if (peek() != c) fail(std::string("expected `") + c + "`");
        ++at_;
    }
    bool word(const char* w) {
        const size_t k = strlen(w);
        if (n_ - at_ < k || memcmp(p_ + at_, w, k) != 0) return false;
        at_ += k;
        return true;
    }

    Json value(const std::string& where, int depth) {
        if (depth > 64) fail("nested too deeply");
        Json v;
        v.where_ = where;
        const char c = peek();
        if (c == '{') {
            v.kind_ = Json::Object;
            ++at_;
            if (peek() == '}') { ++at_; return v; }
            for (;;) {
                if (peek() != '"') fail("expected a member name");
                const std::string key = string();
                expect(':');
                Json m = value(where + "." + key, depth + 1);
                if (!v.members_.emplace(key, std::move(m)).second) fail("duplicate member `" + key + "`");
                if (peek() == ',') { ++at_; continue; }
                expect('}');
                return v;
            }
        }
        if (c == '[') {
            v.kind_ = Json::Array;
            ++at_;
            if (peek() == ']') { ++at_; return v; }
            for (;;) {
                v.items_.push_back(value(where + "[" + std::to_string(v.items_.size()) + "]", depth + 1));
                if (peek() == ',') { ++at_; continue; }
                expect(']');
                return v;
            }
        }
        if (c == '"') {
            v.kind_ = Json::String;
            v.str_ = string();
            return v;
        }
        if (word("true")) { v.kind_ = Json::Bool; v.bool_ = true; return v; }
        if (word("false")) { v.kind_ = Json::Bool; return v; }
        if (word("null")) return v;
        number(v);
        return v;
    }

    void number(Json& v) {
        size_t e = at_;
        bool integral = true;
        while (e < n_ && (isdigit((unsigned char)p_[e]) || strchr("+-.eE", p_[e]) != nullptr) && p_[e] != 0) {
            if (p_[e] == '.' || p_[e] == 'e' || p_[e] == 'E') integral = false;
            ++e;
        }
        const std::string s(p_ + at_, e - at_);
        char* end = nullptr;
        v.num_ = strtod(s.c_str(), &end);
        if (s.empty() || *end != 0 || !std::isfinite(v.num_)) fail("expected a value");
        v.kind_ = Json::Number;
        v.integral_ = integral && std::fabs(v.num_) < 9.0e18;
        if (v.integral_) v.int_ = strtoll(s.c_str(), nullptr, 10);
        at_ = e;
    }

    std::string string() {
        ++at_;  // the opening quote
        std::string out;
        for (;;) {
            if (at_ >= n_) fail("unterminated string");
            const char c = p_[at_++];
            if (c == '"') return out;
            if (c != '\\') { out.push_back(c); continue; }
            if (at_ >= n_) fail("unterminated string");
            const char e = p_[at_++];
            switch (e) {
                case 'n': out.push_back('\n'); break;
                case 't': out.push_back('\t'); break;
                case 'r': out.push_back('\r'); break;
                case 'b': out.push_back('\b'); break;
                case 'f': out.push_back('\f'); break;
                case '"': case '\\': case '/': out.push_back(e); break;
                case 'u': {
                    if (n_ - at_ < 4) fail("short \\u escape");
                    const std::string hex(p_ + at_, 4);
                    char* end = nullptr;
                    const unsigned long cp = strtoul(hex.c_str(), &end, 16);
                    if (*end != 0) fail("bad \\u escape");
                    at_ += 4;
                    if (cp < 0x80) {
                        out.push_back((char)cp);
                    } else if (cp < 0x800) {
                        out.push_back((char)(0xC0 | (cp >> 6)));
                        out.push_back((char)(0x80 | (cp & 0x3F)));
                    } else {
                        out.push_back((char)(0xE0 | (cp >> 12)));
                        out.push_back((char)(0x80 | ((cp >> 6) & 0x3F)));
                        out.push_back((char)(0x80 | (cp & 0x3F)));
                    }
                    break;
                }
                default: fail("unknown escape");
            }
        }
    }

    const char* p_;
    size_t n_, at_ = 0;
    std::string what_;
};

Json Json::parse(const char* text, size_t n, const std::string& what) { return JsonReader(text, n, what).document(); }

const std::map<std::string, Json>& Json::members() const {
    if (kind_ != Object) throw std::runtime_error(where_ + " must be an object");
    return members_;
}

const std::vector<Json>& Json::items() const {
    if (kind_ != Array) throw std::runtime_error(where_ + " must be an array");
    return items_;
}

const Json* Json::find(const std::string& key) const {
    const auto& m = members();
    auto it = m.find(key);
    return it == m.end() ? nullptr : &it->second;
}

const Json& Json::at(const std::string& key) const {
    const Json* v = find(key);
    if (v == nullptr) throw std::runtime_error(where_ + "." + key + " is missing");
    return *v;
}

const std::string& Json::str() const {
    if (kind_ != String) throw std::runtime_error(where_ + " must be a string");
    return str_;
}

double Json::number() const {
    if (kind_ != Number) throw std::runtime_error(where_ + " must be a number");
    return num_;
}

int64_t Json::integer() const {
    if (kind_ != Number) throw std::runtime_error(where_ + " must be a number");
    if (integral_) return int_;
    if (num_ != std::floor(num_) || std::fabs(num_) > 9.0e15) throw std::runtime_error(where_ + " must be an integer");
    return (int64_t)num_;
}

}  // namespace mk
